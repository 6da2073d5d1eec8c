"""Latent attention (`lm.hybrid.LatentSpec`) on the engine: packed weights, the latent cache, and the forms a step can take.

A token's cache row is [latent | rotated key part], zero-padded to a multiple of 64 columns, shared by all heads.
Queries can meet it in two ways that give the same sums:

* absorbed: W_uk goes to the query side, q_lat = W_uk^T q, and the scores are products with the cache rows themselves; the
  weighted latents go through W_uv.  Nothing per key is formed, so this is the form of decoding and of short segments.
* expanded: keys and values of every head are formed from the latents with one product.  Per score it is several times
  cheaper (dim + rope_dims + vdim columns instead of 2 kv_rank + rope_dims), so long segments take it.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..lm.hybrid import LatentSpec
from .prompt import StepPlan, Window


def _pad(n: int, to: int) -> int:
    return (n + to - 1) // to * to


class LatentShape:
    """Padded sizes of one layer."""

    def __init__(self, m: LatentSpec):
        self.dim, self.rot = _pad(m.dim, 16), _pad(m.rope_dims, 16)
        self.vdim, self.rank = _pad(m.vdim, 8), _pad(m.kv_rank, 16)
        self.head = self.dim + self.rot          # columns of a query head
        self.row = _pad(self.rank + self.rot, 64)     # columns of a cache row


def check(engine, i: int, m: LatentSpec) -> None:
    from ..ops import _mixers as M
    s = LatentShape(m)
    if engine.fast and (s.rank > M.LATENT_MAX_RANK or s.row > M.LATENT_MAX_ROW):
        raise ValueError(f"layer {i}: the BF16 kernels take latents of up to {M.LATENT_MAX_RANK} columns, cache rows of up to "
                         f"{M.LATENT_MAX_ROW}")
    if engine.fast and engine.cfg.block_size % 8:
        raise ValueError(f"layer {i}: the BF16 kernels take pages of a multiple of 8 tokens")
    if not engine.fast and s.rank > 1024:
        raise ValueError(f"layer {i}: the FP32 kernel takes latents of up to 1024 columns")


def load(engine, m: LatentSpec, get) -> dict:
    """``get(name)``: the mixer's tensors."""
    s, H = LatentShape(m), m.heads
    dkv = get("dkv")
    out: Dict[str, object] = {"shape": s}
    # queries from the input or from their latent; neighbouring pairs become halves: q and the shared key part, whose products
    # alone matter, are permuted alike
    src = get("uq" if m.q_rank else "q").float()
    src = src.view(H, m.dim + m.rope_dims, src.shape[1])
    order = torch.arange(m.rope_dims)
    if m.interleaved:
        order = order.view(-1, 2).t().reshape(-1)
    wq = torch.zeros((H, s.head, src.shape[2]))
    wq[:, : m.dim], wq[:, s.dim: s.dim + m.rope_dims] = src[:, : m.dim], src[:, m.dim:][:, order]
    wq = wq.view(H * s.head, -1)
    gate = [get("g")] if m.gate else []
    out["in"], off = engine._pack([get("dq") if m.q_rank else wq, dkv[: m.kv_rank], dkv[m.kv_rank:][order], *gate])
    out["off"] = (*off, 0) if not m.gate else tuple(off)
    if m.q_rank:
        out["uq"], _ = engine._pack([wq])
    # [W_uk | W_uv], rows head by head: one product expands a latent; W_uk also serves as [heads, dim, rank]
    ukv = torch.zeros((H * (s.dim + s.vdim), s.rank))
    ukv[: H * s.dim].view(H, s.dim, s.rank)[:, : m.dim, : m.kv_rank] = get("uk").float().view(H, m.dim, m.kv_rank)
    ukv[H * s.dim:].view(H, s.vdim, s.rank)[:, : m.vdim, : m.kv_rank] = get("uv").float().view(H, m.vdim, m.kv_rank)
    out["ukv"], _ = engine._pack([ukv])
    w = out["ukv"].w
    out["uk"], out["uv"] = w[: H * s.dim].view(H, s.dim, s.rank), w[H * s.dim:].view(H, s.vdim, s.rank)
    if engine.fast:                   # the few-rows form wants the summed index last
        out["uk_t"] = out["uk"].transpose(1, 2).contiguous()
        engine.weight_nbytes += out["uk_t"].numel() * out["uk_t"].element_size()
    wo = torch.zeros((engine.d, H, s.vdim))
    wo[:, :, : m.vdim] = get("o").float().view(engine.d, H, m.vdim)
    out["out"], _ = engine._pack([wo.view(engine.d, H * s.vdim)])
    out["w_q"], out["w_kv"] = engine._f32(get("dq.norm")) if m.q_rank else None, engine._f32(get("dkv.norm"))
    out["rope"] = engine._rope_tables(m.rope_dims, m.rope_base, m.rope_scaling)
    return out


FEW_ROWS = 256       # up to this many rows the per-head products stream their weights, above they are batched GEMMs


def _to_latent(engine, lw: dict, q, out) -> None:
    """out[r, h] = q[r, h] W_uk[h] for [rows, heads, .] views."""
    if engine.fast and q.shape[0] <= FEW_ROWS:
        from ..ops import _experts as X
        X.head_product(q, lw["uk_t"], out)
    elif engine.fast:
        from ..ops import _cuda as K
        K.gemm(q.permute(1, 0, 2), lw["uk"], b_mn=True, out=out.permute(1, 0, 2))
    else:
        out.copy_((q.permute(1, 0, 2) @ lw["uk"]).permute(1, 0, 2))


def _from_latent(engine, lw: dict, o, out) -> None:
    """out[r, h] = W_uv[h] o[r, h]."""
    if engine.fast and o.shape[0] <= FEW_ROWS:
        from ..ops import _experts as X
        X.head_product(o, lw["uv"], out)
    elif engine.fast:
        from ..ops import _cuda as K
        K.gemm(o.permute(1, 0, 2), lw["uv"], out=out.permute(1, 0, 2))
    else:
        out.copy_((o.permute(1, 0, 2) @ lw["uv"].transpose(1, 2)).permute(1, 0, 2))


def absorbed(engine, i: int, m: LatentSpec, lw: dict, q, gate, pos, out, groups) -> None:
    """``q`` [rows, heads * head], ``out`` [rows, heads * vdim]; ``groups``: the segments of these rows."""
    from ..ops import _mixers as M
    s, H, n = lw["shape"], m.heads, q.shape[0]
    ql = torch.empty((n, H, s.row), dtype=q.dtype, device=q.device)
    _to_latent(engine, lw, q.view(n, H, s.head)[:, :, : s.dim], ql[:, :, : s.rank])
    ql = ql.view(n, H * s.row)
    M.rope_heads(q, s.head, s.dim, ql, s.row, s.rank, H, m.rope_dims, s.row - s.rank, pos, *lw["rope"])
    ol = torch.empty((n, H * s.rank), dtype=q.dtype, device=q.device)
    for seg in groups:
        if seg.count:
            if engine.fast:
                M.latent_attention(ql, engine.k_cache[i], engine.block_table, ol, seg, heads=H, rank=s.rank, window=m.window,
                                   scale=m.scale, gate=gate, splits=splits(engine, m, seg))
            else:
                M.paged_window_attention(ql, engine.k_cache[i], None, engine.block_table, ol, seg, heads=H,
                                         block_size=engine.cfg.block_size, window=m.window, scale=m.scale, gate=gate, vdim=s.rank)
    _from_latent(engine, lw, ol.view(n, H, s.rank), out.view(n, H, s.vdim))


def splits(engine, m: LatentSpec, seg) -> int:
    """Spans of the keys: enough blocks for every SM, at least 128 keys each."""
    if engine.cfg.decode_splits > 0 and seg.max_len == 1:
        return engine.cfg.decode_splits
    keys = min(m.window, engine.ctx) if m.window > 0 else engine.ctx
    pairs = seg.total * m.heads              # (token, head) rows; a block takes up to 64, of one-token segments one token's
    blocks = seg.count * -(-m.heads // 64) if seg.max_len == 1 else max(seg.count, pairs // 64)
    sms = 296 if seg.max_len == 1 and m.heads <= 16 else 148
    return max(1, min(sms // blocks, -(-keys // 128), 16))


def expandable(m: LatentSpec) -> bool:
    s = LatentShape(m)
    return s.dim <= 128 and s.rot <= 64 and s.vdim <= 128 and m.scale > 0


def expanded(engine, i: int, m: LatentSpec, lw: dict, q, lat, gate, pos, out, step: StepPlan) -> None:
    """The long segments of a step.  ``lat``: latent rows of the step; ``q`` is rotated in place."""
    from ..ops import _mixers as M
    s, w = lw["shape"], Window(m.window)
    if step.gathered:
        lat = torch.empty((step.kv_rows[w], s.row), dtype=engine.adt, device=engine.dev)
        M.latent_gather(engine.k_cache[i], engine.block_table, step.runs[w], step.longest[w], lat)
    kv = engine._linear(lat[:, : s.rank], lw["ukv"])
    M.rope_heads(q, s.head, s.dim, q, s.head, s.dim, m.heads, m.rope_dims, s.rot, pos, *lw["rope"])
    M.latent_prompt(q, kv, lat, out, step.blocks[w], heads=m.heads, dim=s.dim, rot=s.rot, vdim=s.vdim, rank=s.rank, window=w.size,
                    scale=m.scale, gate=gate)


def mixer(engine, i: int, m: LatentSpec, lw: dict, h, pos, slot):
    from ..ops import _mixers as M
    s, n = lw["shape"], h.shape[0]
    step = engine._prompt_plan if expandable(m) else None
    proj = engine._linear(h, lw["in"])
    cq = torch.empty((n, _pad(m.q_rank, 8)), dtype=engine.adt, device=engine.dev) if m.q_rank else None
    gate = torch.empty((n, m.heads), dtype=torch.float32, device=engine.dev) if m.gate else None
    lat = torch.empty((n, s.row), dtype=engine.adt, device=engine.dev) if step is not None and not step.gathered else None
    M.latent_prep(proj, lw["off"], m.q_rank, m.kv_rank, m.rope_dims, m.heads, lw["w_q"], lw["w_kv"], pos, slot, *lw["rope"], cq,
                  engine.k_cache[i], s.rank, gate, eps=engine.model.norm_eps, lat=lat)
    q = engine._linear(cq, lw["uq"]) if m.q_rank else proj[:, : m.heads * s.head]
    out = torch.empty((n, m.heads * s.vdim), dtype=engine.adt, device=engine.dev)
    if step is None:
        groups = [engine._groups[0], engine._many] if engine.fast else [engine._every]
        absorbed(engine, i, m, lw, q, gate, pos, out, groups)
    else:
        if step.rows is not None:       # before the rotation in place
            part = torch.empty((step.rows.shape[0], out.shape[1]), dtype=engine.adt, device=engine.dev)
            absorbed(engine, i, m, lw, q.index_select(0, step.rows), gate.index_select(0, step.rows) if m.gate else None,
                     pos.index_select(0, step.rows), part, step.groups)
        expanded(engine, i, m, lw, q, lat, gate, pos, out, step)
        if step.rows is not None:
            out.index_copy_(0, step.rows, part)
    return engine._linear(out, lw["out"])
