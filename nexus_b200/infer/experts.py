"""Feed-forward of experts (`lm.hybrid.ExpertsSpec`) on the engine.

Where a table picks a token's experts by its id, one launch at the start of a step sorts the assignments of every layer; a
learned router picks and sorts in its layer.  Up to 32 rows per expert the weights are streamed once past all of an expert's
rows; above, the residual kernel (or the routing kernel) writes every row to its slots and the tcgen05 GEMM takes the experts as
groups of row tiles.  The kernel that adds the sublayer's output to the residual stream sums a token's experts, with the
router's weights, and its gated shared expert on the way.

Gated experts keep W_gate and W_up as one matrix in turns of eight rows, so that a unit's gate and value meet in one thread of the
few-rows product and of the GEMM's epilogue."""
from __future__ import annotations

from typing import List, Optional

import torch

from ..lm.hybrid import ExpertsSpec


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _stack(parts) -> torch.Tensor:
    """[experts, rows, columns] zero-padded to multiples of 8."""
    r, c = parts[0].shape
    w = torch.zeros((len(parts), _pad8(r), _pad8(c)))
    for e, p in enumerate(parts):
        w[e, :r, :c] = p.float()
    return w


def in_turns(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """[..., n, k] gates and values as [..., 2 n, k] in turns of eight rows, gates first; n is padded to a multiple of 8."""
    pad = (0, 0, 0, -gate.shape[-2] % 8)
    both = torch.stack([torch.nn.functional.pad(t.float(), pad).unflatten(-2, (-1, 8)) for t in (gate, up)], -3)
    return both.flatten(-4, -2)


def load(engine, f: ExpertsSpec, get) -> dict:
    """``get(name)``: the feed-forward's tensors."""
    out = {}
    if f.router is None:
        out["table"] = get("table").to(engine.dev, torch.int32).contiguous()
    else:
        out["router"], _ = engine._pack([get("router")])
        out["correction"] = engine._f32(get("correction"))
    for name in ("up", "down"):
        w = _stack([get(f"e{e}.{name}") for e in range(f.experts)])
        if f.glu is not None and name == "up":
            w = in_turns(_stack([get(f"e{e}.gate") for e in range(f.experts)]), w)
        out[name] = w.to(engine.dev, engine.adt).contiguous()
        engine.weight_nbytes += out[name].numel() * out[name].element_size()
    if f.shared:
        out["shared_up"], _ = engine._pack([get("shared.up")])
        out["shared_down"], _ = engine._pack([get("shared.down")])
        out["sg"] = engine._f32(get("shared.sg").reshape(-1))
    return out


def alignment(engine, f: ExpertsSpec, rows: int) -> int:
    """Slots an expert's rows are padded to, which also picks the product."""
    from ..ops import _experts as X
    if not engine.fast:
        return X.F32_ALIGN
    each = rows * f.top / f.experts
    return 1 if each <= 32 else 128 if each < 640 else 256


def route(engine, tok) -> List[Optional[object]]:
    """A `Route` for every layer whose experts a table picks."""
    from ..ops import _experts as X
    routes: List[Optional[object]] = [None] * engine.L
    by_align = {}
    for i, layer in enumerate(engine.runs):
        if layer.experts is not None and layer.experts.router is None:
            by_align.setdefault(alignment(engine, layer.experts, tok.shape[0]), []).append(i)
    for align, which in by_align.items():
        got = X.table_route(tok, [(engine.layers[i]["ff"]["table"], engine.runs[i].experts.experts) for i in which], align)
        for i, r in zip(which, got):
            routes[i] = r
    return routes


def gate(engine, f: ExpertsSpec, lw: dict, h):
    """The `Route` of the router's choices for the rows ``h``, and the rows in slot order where the GEMM wants them."""
    from ..ops import _experts as X
    align = alignment(engine, f, h.shape[0])
    logits = engine._linear(h, lw["router"], out_dtype=torch.float32)
    return X.gate_route(logits, lw["correction"], f.top, align, n_groups=f.router.groups, keep=f.router.keep,
                        h=h if align >= 128 else None)


def forward(engine, f: ExpertsSpec, lw: dict, r, h, sorted_h):
    """``h``: the rows of the batch; ``sorted_h``: the same in slot order (GEMM form) or None.  Returns the experts' rows in
    slot order and the shared expert's output (or None)."""
    from ..ops import _experts as X
    from ..ops import _mixers as M
    gather = sorted_h is None
    act = {"act": "relu2"} if f.glu is None else {"gate": M.Glu(2, f.glu.limit, f.glu.slope, f.glu.offset)}
    a = X.expert_product(h if gather else sorted_h, lw["up"], r, gather=gather, **act)
    y = X.expert_product(a, lw["down"], r, gather=False)
    if not f.shared:
        return y, None
    if engine.fast:
        a = engine._linear(h, lw["shared_up"], act="relu2")
    else:
        a = torch.relu(engine._linear(h, lw["shared_up"])).square_()
    return y, engine._linear(a, lw["shared_down"])
