"""Feed-forward of table-routed experts (`lm.hybrid.ExpertsSpec`) on the engine.

Which experts a token uses depends on nothing but its id, so one launch at the start of a step sorts the assignments of
every layer.  Up to 32 rows per expert the weights are streamed once past all of an expert's rows; above, the residual kernel
writes every row to its slots and the tcgen05 GEMM takes the experts as groups of row tiles.  The kernel that adds the
sublayer's output to the residual stream sums a token's experts and its gated shared expert on the way."""
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


def load(engine, f: ExpertsSpec, get) -> dict:
    """``get(name)``: the feed-forward's tensors."""
    out = {"table": get("table").to(engine.dev, torch.int32).contiguous()}
    for name in ("up", "down"):
        out[name] = _stack([get(f"e{e}.{name}") for e in range(f.experts)]).to(engine.dev, engine.adt)
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
    """A `Route` for every layer that has experts."""
    from ..ops import _experts as X
    routes: List[Optional[object]] = [None] * engine.L
    by_align = {}
    for i, layer in enumerate(engine.model.layers):
        if layer.experts is not None:
            by_align.setdefault(alignment(engine, layer.experts, tok.shape[0]), []).append(i)
    for align, which in by_align.items():
        got = X.table_route(tok, [(engine.layers[i]["ff"]["table"], engine.model.layers[i].experts.experts) for i in which], align)
        for i, r in zip(which, got):
            routes[i] = r
    return routes


def forward(engine, f: ExpertsSpec, lw: dict, r, h, sorted_h):
    """``h``: the rows of the batch; ``sorted_h``: the same in slot order (GEMM form) or None.  Returns the experts' rows in
    slot order and the shared expert's output (or None)."""
    from ..ops import _experts as X
    gather = sorted_h is None
    a = X.expert_product(h if gather else sorted_h, lw["up"], r, gather=gather, act="relu2")
    y = X.expert_product(a, lw["down"], r, gather=False)
    if not f.shared:
        return y, None
    if engine.fast:
        a = engine._linear(h, lw["shared_up"], act="relu2")
    else:
        a = torch.relu(engine._linear(h, lw["shared_up"])).square_()
    return y, engine._linear(a, lw["shared_down"])
