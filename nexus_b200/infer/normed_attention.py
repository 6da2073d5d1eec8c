"""Attention on normed queries and keys (`lm.hybrid.NormedAttentionSpec`) on the engine.

One projection gives q, k, v and the output gate; one kernel norms q and k (and v), applies every factor of the scores to q (scale,
the head's factor, the position's temperature), appends k and v to the cache pages and takes the gate's sigmoid.  Heads are
zero-padded to sizes the kernels load in whole vectors; norms count the real columns.

Heads that mix their weights after the softmax.  out_h = sum_g T[h, g] (P_g V of the KV head of h), so:

* decoding and short segments: scores of all heads, then the mixture of the normalised weights, then one product per KV head with its
  values;
* longer segments and FP32: every head's weights meet the values of every KV head inside the attention kernel, and the mixture is taken
  over those outputs."""
from __future__ import annotations

import torch

from ..lm.hybrid import NormedAttentionSpec
from .conv_attention import _pad, _pad_heads
from .prompt import Window


class NormedAttentionShape:
    """Padded sizes of one layer."""

    def __init__(self, m: NormedAttentionSpec):
        self.dim, self.vdim = _pad(m.dim, 16), _pad(m.vdim, 8)
        self.q, self.k, self.v = m.heads * self.dim, m.kv_heads * self.dim, m.kv_heads * self.vdim
        self.offsets = (0, self.q, self.q + self.k, self.q + self.k + self.v)      # q, k, v, gate


def check(engine, i: int, m: NormedAttentionSpec) -> None:
    from ..ops import _mixers as M
    s = NormedAttentionShape(m)
    if engine.fast and max(s.dim, s.vdim) > 256:
        raise ValueError(f"layer {i}: the BF16 attention kernels take head sizes up to 256")
    if not engine.fast and s.vdim > 1024:
        raise ValueError(f"layer {i}: the FP32 kernel takes value sizes up to 1024")
    if m.talk and m.heads > M.TALK_MAX_HEADS:
        raise ValueError(f"layer {i}: up to {M.TALK_MAX_HEADS} heads mix their weights")


def load(engine, m: NormedAttentionSpec, get) -> dict:
    """``get(name)``: the mixer's tensors."""
    from ..ops import _mixers as M
    s = NormedAttentionShape(m)
    parts = (("q", m.heads, s.dim), ("k", m.kv_heads, s.dim), ("v", m.kv_heads, s.vdim))

    def stack(suffix):
        return torch.cat([_pad_heads(get(n + suffix), heads, size) for n, heads, size in parts], 0)
    out = {"shape": s}
    w = torch.cat([stack("")] + ([get("g").float()] if m.gate else []), 0)
    w = torch.nn.functional.pad(w, (0, 0, 0, -w.shape[0] % 64))      # rows of the projection start on 128 bytes, as the tiles read from them
    out["in"], _ = engine._pack([w], bias=stack(".b") if m.bias else None)
    wo = torch.zeros((engine.d, m.heads, s.vdim))
    wo[:, :, : m.vdim] = get("o").float().view(engine.d, m.heads, m.vdim)
    out["out"], _ = engine._pack([wo.view(engine.d, m.heads * s.vdim)], bias=get("o.b") if m.bias else None)
    for n, heads in (("q", m.heads), ("k", m.kv_heads)):
        out[n + "_norm"] = engine._f32(_pad_heads(get(n + ".norm"), heads if m.norm == "all" else 1, s.dim))
    out["head_scale"] = engine._f32(get("temp")) if m.head_scale else None
    out["talk"] = engine._f32(get("talk")) if m.talk else None
    out["bias"] = out["bias_wide"] = None
    if m.distance is not None:      # one entry per distance; the last one counts for all beyond
        rows = [m.distance.bucket(n) for n in range(m.distance.far + 1)]
        while len(rows) > 1 and rows[-1] == rows[-2]:
            rows.pop()
        out["bias"] = engine._f32(get("rel").float()[rows].t())
        if promptable(m):
            out["bias_wide"] = M.extended_bias(out["bias"])
    return out


def alloc(engine, i: int, m: NormedAttentionSpec) -> None:
    s, cfg = NormedAttentionShape(m), engine.cfg
    for cache, size in ((engine.k_cache, s.dim), (engine.v_cache, s.vdim)):
        cache[i] = torch.zeros((engine.n_blocks, cfg.block_size, m.kv_heads, size), dtype=engine.adt, device=engine.dev)


def window(m: NormedAttentionSpec) -> Window:
    return Window(m.window, 0, m.chunk)


def promptable(m: NormedAttentionSpec) -> bool:
    """Whether the tcgen05 prompt kernel has this layer's sizes."""
    from ..ops import _mixers as M
    s = NormedAttentionShape(m)
    return s.dim <= 128 and s.vdim <= 128 and m.softcap == 0 and (m.distance is None or m.distance.far < M.PROMPT_MAX_BIAS)


def slices(mixers) -> dict:
    """The most rows that layers of heads that mix take at once, by window."""
    from ..ops import _mixers as M
    out: dict = {}
    for m in mixers:
        if isinstance(m, NormedAttentionSpec) and m.talk and promptable(m):
            rows = M.talk_rows(m.heads, m.kv_heads, NormedAttentionShape(m).vdim)
            out[window(m)] = min(rows, out.get(window(m), rows))
    return out


def mixer(engine, i: int, m: NormedAttentionSpec, lw: dict, h, pos, slot):
    from ..ops import _mixers as M
    s, n = lw["shape"], h.shape[0]
    single, short, long_ = engine._groups
    step = engine._prompt_plan if promptable(m) else None
    proj = engine._linear(h, lw["in"])
    gate = torch.empty((n, m.heads), dtype=torch.float32, device=engine.dev) if m.gate else None
    temp = m.temperature
    M.head_prep(proj, s.offsets, heads=m.heads, kv_heads=m.kv_heads, dim=s.dim, vdim=s.vdim, norm_dim=m.dim, norm_vdim=m.vdim,
                norm_all=m.norm == "all", unit_values=m.unit_values, store_kv=step is not None and not step.gathered,
                eps=engine.model.norm_eps, q_scale=m.scale, head_scale=lw["head_scale"], coef=temp.coef if temp else 0.0,
                every=temp.every if temp else 0, w_q=lw["q_norm"], w_k=lw["k_norm"], positions=pos, slots=slot,
                k_cache=engine.k_cache[i], v_cache=engine.v_cache[i], gate=gate)
    q = proj[:, : s.q]
    out = torch.empty((n, m.heads * s.vdim), dtype=engine.adt, device=engine.dev)
    kw = dict(heads=m.heads, block_size=engine.cfg.block_size, window=m.window, chunk=m.chunk, scale=1.0, softcap=m.softcap,
              bias=lw["bias"])
    paged = (engine.k_cache[i], engine.v_cache[i], engine.block_table)
    sizes = dict(heads=m.heads, kv_heads=m.kv_heads, vdim=s.vdim)

    def keys_of_step():
        w = window(m)
        if not step.gathered:
            return (proj[:, o: o + cols] for o, cols in zip(s.offsets[1:3], (s.k, s.v)))
        k, v = (torch.empty((step.kv_rows[w], cols), dtype=engine.adt, device=engine.dev) for cols in (s.k, s.v))
        for c, dst in ((engine.k_cache[i], k), (engine.v_cache[i], v)):
            M.latent_gather(c, engine.block_table, step.runs[w], step.longest[w], dst)
        return k, v
    if m.talk:
        if step is not None:
            M.talk_prompt_mixed(q, *keys_of_step(), out, step.slices[window(m)], lw["talk"], gate, dim=s.dim, window=m.window, chunk=m.chunk,
                                scale=1.0, bias=lw["bias_wide"], distances=lw["bias"].shape[1] if lw["bias"] is not None else 0, **sizes)
        elif not engine.fast or long_.count:
            wide = torch.empty((n, m.heads * m.kv_heads * s.vdim), dtype=engine.adt, device=engine.dev)
            M.paged_window_attention(q, *paged, wide, long_ if engine.fast else engine._every, all_values=True, **kw)
            M.head_mix(wide, lw["talk"], gate, out, **sizes)
        for seg in (single, short) if engine.fast else ():       # after the mixture, which wrote rows between the long segments
            if seg.count:
                M.talk_paged(q, *paged, out, lw["talk"], seg, keys=engine._most_keys(m), splits=engine._decode_splits(m, seg.count),
                             gate=gate, **kw)
        return engine._linear(out, lw["out"])

    def attend(seg, **more):
        if seg.count:
            M.paged_window_attention(q, *paged, out, seg, gate=gate, **kw, **more)
    if not engine.fast:
        attend(engine._every)
        return engine._linear(out, lw["out"])
    attend(single, splits=engine._decode_splits(m, single.count))
    if step is None:
        attend(engine._many)
    else:
        attend(short)
        M.window_prompt(q, *keys_of_step(), out, step.blocks[window(m)], dim=s.dim, window=m.window, chunk=m.chunk, scale=1.0,
                        bias=lw["bias"], gate=gate, **sizes)
    return engine._linear(out, lw["out"])
