"""Latent attention (`lm.hybrid.LatentSpec`) on the engine: packed weights, the latent cache, and the forms a step can take.

A token's cache row is [latent | rotated key part], each part zero-padded to a multiple of 16 columns, shared by all heads.
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


def _pad(n: int, to: int) -> int:
    return (n + to - 1) // to * to


class LatentShape:
    """Padded sizes of one layer."""

    def __init__(self, m: LatentSpec):
        self.dim, self.rot = _pad(m.dim, 16), _pad(m.rope_dims, 16)
        self.vdim, self.rank = _pad(m.vdim, 8), _pad(m.kv_rank, 16)
        self.head = self.dim + self.rot          # columns of a query head
        self.row = self.rank + self.rot          # columns of a cache row


def load(engine, m: LatentSpec, get) -> dict:
    """``get(name)``: the mixer's tensors."""
    s, H = LatentShape(m), m.heads
    dkv = get("dkv")
    out: Dict[str, object] = {"shape": s}
    out["in"], out["off"] = engine._pack([get("dq"), dkv[: m.kv_rank], dkv[m.kv_rank:], get("g")])
    uq = torch.zeros((H, s.head, m.q_rank))
    src = get("uq").float().view(H, m.dim + m.rope_dims, m.q_rank)
    uq[:, : m.dim], uq[:, s.dim: s.dim + m.rope_dims] = src[:, : m.dim], src[:, m.dim:]
    out["uq"], _ = engine._pack([uq.view(H * s.head, m.q_rank)])
    # [W_uk | W_uv], rows head by head: one product expands a latent; W_uk also serves as [heads, dim, rank]
    ukv = torch.zeros((H * (s.dim + s.vdim), s.rank))
    ukv[: H * s.dim].view(H, s.dim, s.rank)[:, : m.dim, : m.kv_rank] = get("uk").float().view(H, m.dim, m.kv_rank)
    ukv[H * s.dim:].view(H, s.vdim, s.rank)[:, : m.vdim, : m.kv_rank] = get("uv").float().view(H, m.vdim, m.kv_rank)
    out["ukv"], _ = engine._pack([ukv])
    w = out["ukv"].w
    out["uk"], out["uv"] = w[: H * s.dim].view(H, s.dim, s.rank), w[H * s.dim:].view(H, s.vdim, s.rank)
    wo = torch.zeros((engine.d, H, s.vdim))
    wo[:, :, : m.vdim] = get("o").float().view(engine.d, H, m.vdim)
    out["out"], _ = engine._pack([wo.view(engine.d, H * s.vdim)])
    out["w_q"], out["w_kv"] = engine._f32(get("dq.norm")), engine._f32(get("dkv.norm"))
    out["rope"] = engine._rope_tables(m.rope_dims, m.rope_base, m.rope_scaling)
    return out


def _per_head(engine, a, b, out, b_mn: bool) -> None:
    """out[h] = a[h] b[h]^T (``b_mn``: a[h] b[h]) for strided batches of matrices."""
    if engine.fast:
        from ..ops import _cuda as K
        K.gemm(a, b, b_mn=b_mn, out=out)
    else:
        out.copy_(a @ (b if b_mn else b.transpose(1, 2)))


def absorbed(engine, i: int, m: LatentSpec, lw: dict, q, gate, pos, out, groups) -> None:
    """``q`` [rows, heads * head], ``out`` [rows, heads * vdim]; ``groups``: the segments of these rows."""
    from ..ops import _mixers as M
    s, H, n = lw["shape"], m.heads, q.shape[0]
    ql = torch.empty((n, H, s.row), dtype=q.dtype, device=q.device)
    _per_head(engine, q.view(n, H, s.head)[:, :, : s.dim].permute(1, 0, 2), lw["uk"], ql[:, :, : s.rank].permute(1, 0, 2), True)
    ql = ql.view(n, H * s.row)
    M.rope_heads(q, s.head, s.dim, ql, s.row, s.rank, H, m.rope_dims, s.rot, pos, *lw["rope"])
    ol = torch.empty((n, H * s.rank), dtype=q.dtype, device=q.device)
    for seg in groups:
        if seg.count:
            M.paged_window_attention(ql, engine.k_cache[i], None, engine.block_table, ol, seg, heads=H,
                                     block_size=engine.cfg.block_size, window=m.window, scale=m.scale, gate=gate, vdim=s.rank,
                                     splits=splits(engine, m, seg.count))
    _per_head(engine, ol.view(n, H, s.rank).permute(1, 0, 2), lw["uv"], out.view(n, H, s.vdim).permute(1, 0, 2), False)


def splits(engine, m: LatentSpec, rows: int) -> int:
    if engine.cfg.decode_splits > 0:
        return engine.cfg.decode_splits
    keys = min(m.window, engine.ctx) if m.window > 0 else engine.ctx
    ctas = rows * (-(-m.heads // 16))
    return max(1, min(296 // max(ctas, 1), -(-keys // 128), 32))


def mixer(engine, i: int, m: LatentSpec, lw: dict, h, pos, slot):
    from ..ops import _mixers as M
    s, n = lw["shape"], h.shape[0]
    proj = engine._linear(h, lw["in"])
    cq = torch.empty((n, _pad(m.q_rank, 8)), dtype=engine.adt, device=engine.dev)
    gate = torch.empty((n, m.heads), dtype=torch.float32, device=engine.dev)
    M.latent_prep(proj, lw["off"], m.q_rank, m.kv_rank, m.rope_dims, m.heads, lw["w_q"], lw["w_kv"], pos, slot, *lw["rope"], cq,
                  engine.k_cache[i], s.rank, gate, eps=engine.model.norm_eps)
    q = engine._linear(cq, lw["uq"])
    out = torch.empty((n, m.heads * s.vdim), dtype=engine.adt, device=engine.dev)
    groups = [engine._every] if not engine.fast else [engine._groups[0], engine._many]
    absorbed(engine, i, m, lw, q, gate, pos, out, groups)
    return engine._linear(out, lw["out"])
