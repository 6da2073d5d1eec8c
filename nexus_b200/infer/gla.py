"""Gated linear attention (`lm.hybrid.GlaSpec`) on the engine: one projection for q, k, v, the output gate and the first decay
projection; the second decay projection and the logarithm of the decays in one kernel; then the recurrence."""
from __future__ import annotations

import torch

from ..lm.hybrid import GlaSpec


def load(engine, m: GlaSpec, get) -> dict:
    """``get(name)``: the mixer's tensors."""
    out = {}
    out["in"], out["off"] = engine._pack([get(n) for n in ("q", "k", "v", "g", "a1")])
    out["out"], _ = engine._pack([get("o")])
    out["a2"], out["a2_b"], out["norm"] = engine._f32(get("a2")), engine._f32(get("a2.b")), engine._f32(get("norm"))
    return out


def parts(engine, m: GlaSpec) -> int:
    """Spans per long segment: enough (segment, head, column tile, span) blocks to fill the GPU, at least 4 chunks each."""
    seg = engine._groups[2]
    blocks = seg.count * m.heads * -(-m.vdim // 64)
    return max(1, min(296 // max(1, blocks), -(-seg.max_len // 64) // 4))


def mixer(engine, i: int, m: GlaSpec, lw: dict, h):
    from ..ops import _mixers as M
    n, qk, vv = h.shape[0], m.heads * m.dim, m.heads * m.vdim
    proj = engine._linear(h, lw["in"])
    oq, ok, ov, og, oa = lw["off"]
    decay = M.decay_gate(proj[:, oa: oa + m.rank], lw["a2"], lw["a2_b"], m.tau)
    o = torch.empty((n, vv), dtype=engine.adt, device=engine.dev)
    args = (proj[:, oq: oq + qk], proj[:, ok: ok + qk], proj[:, ov: ov + vv], decay, o, engine.state[i])
    stepped, chunked = engine._recurrence_groups(m.dim)
    if stepped.count:
        M.gla(*args, stepped, q_scale=m.dim ** -0.5)
    if chunked is not None:
        M.gla(*args, chunked, q_scale=m.dim ** -0.5, chunked=True, parts=parts(engine, m))
    out = engine._buffer(n, vv)
    M.gated_norm(o, proj[:, og: og + vv], lw["norm"], out[:, :vv], groups=m.heads, gate_first=False, eps=engine.model.norm_eps)
    return engine._linear(out, lw["out"])
