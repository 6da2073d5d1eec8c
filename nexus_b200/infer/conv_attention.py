"""Attention over convolved projections (`lm.hybrid.ConvAttentionSpec`) on the engine.

One projection gives q, k and v; one kernel runs the short convolution over its columns, rotates q and k, mixes the values with
those of the first layer that mixes, and appends k and v to the cache pages.  Heads are zero-padded to sizes the kernels load in
whole vectors.  What a sequence owns beside its pages are the last inputs of the convolution."""
from __future__ import annotations

import torch

from ..lm.hybrid import ConvAttentionSpec
from .prompt import Window


def _pad(n: int, to: int) -> int:
    return (n + to - 1) // to * to


class ConvAttentionShape:
    """Padded sizes of one layer."""

    def __init__(self, m: ConvAttentionSpec):
        self.dim, self.vdim = _pad(m.dim, 16), _pad(m.vdim, 8)
        self.q, self.k, self.v = m.heads * self.dim, m.kv_heads * self.dim, m.kv_heads * self.vdim
        self.channels = self.q + self.k + self.v


def check(engine, i: int, m: ConvAttentionSpec) -> None:
    s = ConvAttentionShape(m)
    if engine.fast and max(s.dim, s.vdim) > 256:
        raise ValueError(f"layer {i}: the BF16 attention kernels take head sizes up to 256")
    if not engine.fast and s.vdim > 1024:
        raise ValueError(f"layer {i}: the FP32 kernel takes value sizes up to 1024")


def _pad_heads(t: torch.Tensor, heads: int, size: int) -> torch.Tensor:
    """[heads * n, ...] -> [heads * size, ...], zeros behind every head."""
    t = t.float().reshape(heads, -1, *t.shape[1:])
    out = torch.zeros((heads, size, *t.shape[2:]))
    out[:, : t.shape[1]] = t
    return out.reshape(heads * size, *t.shape[2:])


def load(engine, m: ConvAttentionSpec, get) -> dict:
    """``get(name)``: the mixer's tensors."""
    s = ConvAttentionShape(m)
    parts = (("q", m.heads, s.dim), ("k", m.kv_heads, s.dim), ("v", m.kv_heads, s.vdim))

    def stack(suffix):
        return torch.cat([_pad_heads(get(n + suffix), heads, size) for n, heads, size in parts], 0)
    out = {"shape": s}
    out["in"], _ = engine._pack([stack("")], bias=stack(".b") if m.bias else None)
    out["conv"] = engine._f32(stack(".conv").t())
    wo = torch.zeros((engine.d, m.heads, s.vdim))
    wo[:, :, : m.vdim] = get("o").float().view(engine.d, m.heads, m.vdim)
    out["out"], _ = engine._pack([wo.view(engine.d, m.heads * s.vdim)])
    out["sink"] = engine._f32(get("sink")) if m.sink else None
    out["mix"] = engine._f32(get("vmix").reshape(1)) if m.mix_values else None
    out["rope"] = engine._rope_tables(m.rope_dims, m.rope_base)
    return out


def alloc(engine, i: int, m: ConvAttentionSpec) -> None:
    s, cfg = ConvAttentionShape(m), engine.cfg
    for cache, size in ((engine.k_cache, s.dim), (engine.v_cache, s.vdim)):
        cache[i] = torch.zeros((engine.n_blocks, cfg.block_size, m.kv_heads, size), dtype=engine.adt, device=engine.dev)
    engine.conv_tail[i] = torch.zeros((cfg.max_seqs, max(m.conv - 1, 1), s.channels), dtype=engine.adt, device=engine.dev)


def window(m: ConvAttentionSpec) -> Window:
    return Window(m.window, m.keep_first if m.window > 0 else 0)


def promptable(m: ConvAttentionSpec) -> bool:
    """Whether the tcgen05 prompt kernel has this layer's sizes."""
    s = ConvAttentionShape(m)
    return s.dim <= 128 and s.vdim <= 128 and m.scale > 0 and m.softcap == 0


def mixer(engine, i: int, m: ConvAttentionSpec, lw: dict, h, slot):
    from ..ops import _mixers as M
    s, n = lw["shape"], h.shape[0]
    single, short, long_ = engine._groups
    step = engine._prompt_plan if promptable(m) else None
    proj = engine._linear(h, lw["in"])
    y = torch.empty((n, s.channels), dtype=engine.adt, device=engine.dev)
    mix = None
    if m.mix_values:
        if i == engine.model.first_mixing:
            engine._first_values = torch.empty((n, s.v), dtype=engine.adt, device=engine.dev)
        else:
            mix = lw["mix"]
    cache = dict(k_cache=engine.k_cache[i], v_cache=engine.v_cache[i])
    for seg in (single, engine._many):
        if seg.count:
            M.conv_rope_append(proj, y, lw["conv"], None, engine.conv_tail[i], seg, heads=m.heads, kv_heads=m.kv_heads, dim=s.dim,
                               vdim=s.vdim, rot_dims=m.rope_dims, cos_t=lw["rope"][0], sin_t=lw["rope"][1], slots=slot,
                               store_kv=step is not None and not step.gathered, mix=mix,
                               first=engine._first_values if m.mix_values else None, **cache)
    q = y[:, : s.q]
    out = torch.empty((n, m.heads * s.vdim), dtype=engine.adt, device=engine.dev)

    def paged(seg, **kw):
        if seg.count:
            M.paged_window_attention(q, engine.k_cache[i], engine.v_cache[i], engine.block_table, out, seg, heads=m.heads,
                                     block_size=engine.cfg.block_size, window=m.window, keep_first=m.keep_first, scale=m.scale,
                                     softcap=m.softcap, sink=lw["sink"], **kw)
    if not engine.fast:
        paged(engine._every)
        return engine._linear(out, lw["out"])
    paged(single, splits=engine._decode_splits(m, single.count))
    if step is None:
        paged(engine._many)
        return engine._linear(out, lw["out"])
    paged(short)
    w = window(m)
    if step.gathered:
        k, v = (torch.empty((step.kv_rows[w], cols), dtype=engine.adt, device=engine.dev) for cols in (s.k, s.v))
        for c, dst in ((engine.k_cache[i], k), (engine.v_cache[i], v)):
            M.latent_gather(c, engine.block_table, step.runs[w], step.longest[w], dst)
    else:
        k, v = y[:, s.q: s.q + s.k], y[:, s.q + s.k:]
    M.window_prompt(q, k, v, out, step.blocks[w], heads=m.heads, kv_heads=m.kv_heads, dim=s.dim, vdim=s.vdim, window=w.size,
                    scale=m.scale, keep_first=w.keep_first, kept=step.kept[w], sink=lw["sink"])
    return engine._linear(out, lw["out"])
