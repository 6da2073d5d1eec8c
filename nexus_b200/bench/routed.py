"""Serving speed of a Gutivik model beside the framework's other models of the same width and depth, and the roofline of its
kernels.

    python -m nexus_b200.bench.routed [--sizes 1024,2048,4096] [--kernels] [--peaks MEASURED_PEAKS.json] [--only REGEX]

The measurements are those of `bench.hybrid` (packed prefill of fresh prompts, captured decode steps of 64 sequences with
1024 tokens behind them, kernels with a cold L2 against the measured peaks)."""
from __future__ import annotations

import argparse
import json
import re
import sys

import torch

from .hybrid import SIZES, VOCAB, hybrid_config, time_engine


def routed_config(width: int, layers: int, dim: int):
    """Attention, gated linear attention and latent attention in turn; window 1024, 4 query heads to a KV head, 16 kept first keys;
    32 gated experts of width / 2 in 4 groups of which a token uses 4 from 2 groups, a dense feed-forward in the first layer."""
    from ..lm.hybrid import (ClampedGlu, ConvAttentionSpec, ExpertsSpec, GlaSpec, HybridConfig, HybridLayer, LatentSpec, RouterSpec)
    heads = width // dim
    mixers = (ConvAttentionSpec(heads, heads // 4, dim, dim, dim ** -0.5, 0.0, 1024, dim // 2, 250000.0, conv=4, keep_first=16,
                                mix_values=True),
              GlaSpec(width // 128, 64, 128, 16.0, 16),
              LatentSpec(width // 128, 128, 64, 128, 0, 512, 192 ** -0.5, 1024, 10000.0, interleaved=True, gate=False))
    experts = ExpertsSpec(32, 4, width // 2, router=RouterSpec(4, 2), glu=ClampedGlu(7.0))
    out = [HybridLayer(mixers[0], ff=width * 2, act="gelu_tanh")]
    out += [HybridLayer(mixers[i % 3], experts=experts) for i in range(1, layers)]
    return HybridConfig(VOCAB, width, out, 1e-5, logit_softcap=30.0, name=f"gutivik-{width}", post_norm=False, norm_offset=1.0,
                        logit_scale=2.0)


def active_parameters(cfg) -> int:
    """Weights one token meets (embedding row aside)."""
    from ..lm.gutivik import gutivik_tensors
    n = 0
    for name, shape in gutivik_tensors(cfg).items():
        part = name.split(".")
        if name == "embed":
            continue
        size = 1
        for s in shape:
            size *= s
        if len(part) > 2 and part[1] == "mlp" and part[2][0] == "e" and part[2][1:].isdigit():
            f = cfg.layers[int(part[0][1:])].experts
            size = size * f.top // f.experts
        n += size
    return n


def model_lines(sizes, iters=10):
    from ..infer import Gpt2Weights
    from ..lm.gutivik import random_gutivik
    from ..lm.hybrid import random_gugedra
    from ..lm.makuzen import random_makuzen
    from .latent import latent_config
    rows = []
    for width in sizes:
        layers, dim = SIZES[width]
        cfg = routed_config(width, layers, dim)
        gt = time_engine(random_gutivik(cfg), iters=iters)
        gt["active_parameters"] = active_parameters(cfg)
        mk = time_engine(random_makuzen(latent_config(width, layers)), iters=iters)
        gu = time_engine(random_gugedra(hybrid_config(width, layers, dim)), iters=iters)
        gp = time_engine(Gpt2Weights.random(layers, width // dim, width, VOCAB, 4096 + 64), iters=iters)
        rows.append({"width": width, "layers": layers, "gutivik": gt, "makuzen": mk, "gugedra": gu, "gpt2": gp})
    return rows


# ------------------------------------------------------------------------------------------ kernels
def kernel_cases():
    """name -> (launch, flops, bytes)."""
    from ..ops import _cuda as K
    from ..ops import _experts as X
    from ..ops import _mixers as M
    dev, bf, f32 = "cuda", torch.bfloat16, torch.float32
    gen = torch.Generator(device=dev).manual_seed(0)

    def rn(*shape, dtype=bf, s=1.0):
        return (torch.randn(*shape, device=dev, generator=gen) * s).to(dtype)

    def segs(lens, pos):
        t = torch.zeros((4, len(lens)), dtype=torch.int32)
        r = 0
        for i, n in enumerate(lens):
            t[:, i] = torch.tensor([r, n, pos, i], dtype=torch.int32)
            r += n
        return M.Segments(t.to(dev), 0, len(lens), max(lens), r)
    W, N, B, bs, cases = 2048, 8192, 256, 16, {}
    pre, one, long1, short = segs([1024] * 8, 0), segs([1] * B, 1023), segs([N], 0), segs([8] * 32, 1016)
    ones, x, y, h = torch.ones(W, device=dev), rn(N, W, dtype=f32), rn(N, W), rn(N, W)
    E, top, ff = 32, 4, 1024
    corr = rn(E, dtype=f32, s=0.1)
    logits = rn(N, E, dtype=f32)

    def route(n, align, src=None):
        return X.gate_route(logits[:n], corr, top, align, n_groups=4, keep=2, h=src)
    r256, by_slot = route(N, 256, h)
    cases["residual_norm (add, next norm) 8192x2048"] = (lambda: M.residual_norm(x, y=y, w_next=ones, h=h, eps=1e-5), 0, N * W * 12)
    cases["like: residual_norm (post-norm, add, next norm) 8192x2048"] = (
        lambda: M.residual_norm(x, y=y, w_post=ones, w_next=ones, h=h, eps=1e-5), 0, N * W * 12)
    cases["residual_norm + weighted sum of 4 experts 8192x2048"] = (
        lambda: M.residual_norm(x, experts=by_slot, slots=r256.slots, top=top, weights=r256.weight, w_next=ones, h=h, eps=1e-5), 0,
        N * W * (10 + 2 * top))
    cases["like: residual_norm + sum of 4 experts and a shared one 8192x2048"] = (
        lambda: M.residual_norm(x, y=y, w_post=ones, x_cast=h, eps=1e-5, experts=by_slot, slots=r256.slots, top=top), 0,
        N * W * (12 + 2 * top))
    # attention over convolved projections: 32 query heads, 8 KV heads of 64
    H, G, D, win, keep = 32, 8, 64, 1024, 16
    C = (H + 2 * G) * D
    kc, vc = rn(B * 1024 // bs, bs, G, D), rn(B * 1024 // bs, bs, G, D)
    table = torch.randperm(B * 1024 // bs, generator=torch.Generator().manual_seed(1)).view(B, -1).to(torch.int32).to(dev)
    proj, yq, cw, tail = rn(N, C), rn(N, C), rn(4, C, dtype=f32), rn(B, 3, C)
    pos, slot = (torch.arange(N, dtype=torch.int32) % 1024).to(dev), torch.arange(N, dtype=torch.int32, device=dev)
    cos, sin = rn(N, 16, dtype=f32), rn(N, 16, dtype=f32)
    first, lam = rn(N, G * D), torch.full((1,), 0.5, device=dev)
    ck = dict(heads=H, kv_heads=G, dim=D, vdim=D, rot_dims=32, cos_t=cos, sin_t=sin, slots=slot, k_cache=kc, v_cache=vc, first=first, mix=lam)
    cases["conv_rope_append 8192 x (32+8+8) x 64, 4 taps"] = (
        lambda: M.conv_rope_append(proj, yq, cw, None, tail, pre, store_kv=True, **ck), 0, N * (C * 4 + 3 * G * D * 2))
    cases["like: conv_silu 8192 x 3072, 4 taps"] = (lambda: M.conv_silu(proj, yq, cw, None, tail, pre), 0, N * C * 4)
    cases["like: rope_append 8192 x (32+8+8) x 64"] = (
        lambda: M.rope_append(proj, 0, H * D, (H + G) * D, H, G, D, D, 32, pos, slot, cos, sin, kc, vc), 0,
        N * (H * 32 * 4 + G * D * 2 * 4 + G * 32 * 2))
    cases["conv_rope_append decode 256 x 3072"] = (
        lambda: M.conv_rope_append(proj[:B], yq[:B], cw, None, tail, one, **ck), 0, B * (C * 2 * 7 + H * D * 2 + 3 * G * D * 2))
    cases["like: conv_silu decode 256 x 3072"] = (lambda: M.conv_silu(proj[:B], yq[:B], cw, None, tail, one), 0, B * C * 2 * 8)
    sink, out = rn(H, dtype=f32), rn(N, H * D)
    q, k, v = yq[:, : H * D], yq[:, H * D: (H + G) * D], yq[:, (H + G) * D:]

    def blocks(count, length, window):
        back = window - 1 if window else 1 << 30
        b = [(min(p, back) + 256, i * length + p, 256, p, i * length) for i in range(count) for p in range(0, length, 256)]
        b.sort(key=lambda t: -t[0])
        return torch.tensor([t[1:] for t in b], dtype=torch.int32, device=dev)

    def pairs(count, length, window, keep=0):
        return count * sum(min(i + 1, window + min(keep, max(0, i + 1 - window))) if window else i + 1 for i in range(length))
    for count, length in ((8, 1024), (2, 4096)):
        bl = blocks(count, length, win)
        cases[f"window_prompt {count} x {length}, window {win}, 16 kept, sink"] = (
            lambda bl=bl: M.window_prompt(q, k, v, out, bl, heads=H, kv_heads=G, dim=D, vdim=D, window=win, scale=0.125, keep_first=keep,
                                          sink=sink), 4.0 * D * H * pairs(count, length, win, keep), 0)
        q4, k4, v4 = rn(count, length, H, D), rn(count, length, G, D), rn(count, length, G, D)
        cases[f"like: flash {count} x {length}, window {win}"] = (
            lambda q4=q4, k4=k4, v4=v4: K.attention_fwd(q4, k4, v4, window=win), 4.0 * D * H * pairs(count, length, win), 0)
    qd, od = rn(B, H * D), rn(B, H * D)
    pk = dict(heads=H, block_size=bs, window=win, scale=0.125)
    cases["paged_window_decode 256 x 1024, 32 / 8 heads, 16 kept, sink"] = (
        lambda: M.paged_window_attention(qd, kc, vc, table, od, one, keep_first=keep, sink=sink, **pk), 0, B * 1024 * G * D * 4)
    cases["like: paged_window_decode 256 x 1024, 32 / 8 heads"] = (
        lambda: M.paged_window_attention(qd, kc, vc, table, od, one, **pk), 0, B * 1024 * G * D * 4)
    cases["paged_window_prefill, 32 portions of 8 behind 1016, kept, sink"] = (
        lambda: M.paged_window_attention(qd, kc, vc, table, od, short, keep_first=keep, sink=sink, **pk), 4.0 * B * H * D * 1024,
        32 * 1024 * G * D * 4)
    cases["like: paged_window_prefill, 32 portions of 8 behind 1016"] = (
        lambda: M.paged_window_attention(qd, kc, vc, table, od, short, **pk), 4.0 * B * H * D * 1024, 32 * 1024 * G * D * 4)
    # latent attention without a query latent: 16 heads of 128 + 64
    Hl, R, rank, row = 16, 64, 512, 576
    lp, lc, lat = rn(N, Hl * 192 + row), rn(B * 1024 // bs, bs, 1, row), rn(N, row)
    cl, sl, wk = rn(1024, 32, dtype=f32), rn(1024, 32, dtype=f32), torch.ones(rank, device=dev)
    cases["latent_prep 8192 x (512 + 64)"] = (
        lambda: M.latent_prep(lp, (0, Hl * 192, Hl * 192 + rank, 0), 0, rank, R, Hl, None, wk, pos, slot, cl, sl, None, lc, rank, None,
                              eps=1e-5, lat=lat), 0, N * 2 * 3 * row)
    lq, cq, hg, wq = rn(N, 768 + row + Hl), rn(N, 768), torch.rand((N, Hl), device=dev), torch.ones(768, device=dev)
    cases["like: latent_prep 8192 x (768 + 512 + 64 + 16)"] = (
        lambda: M.latent_prep(lq, (0, 768, 768 + rank, 768 + row), 768, rank, R, Hl, wq, wk, pos, slot, cl, sl, cq, lc, rank, hg, eps=1e-5,
                              lat=lat), 0, N * 2 * (2 * 768 + 3 * row + Hl) + N * Hl * 4)
    # gated linear attention: 16 heads, 64 x 128
    Hg, Dk, Dv = 16, 64, 128
    gp, dec, go = rn(N, Hg * (2 * Dk + Dv)), -torch.rand((N, Hg * Dk), device=dev, generator=gen) * 0.3, rn(N, Hg * Dv)
    state = rn(B, Hg, Dk, Dv, dtype=f32)
    gq, gk, gv = gp[:, : Hg * Dk], gp[:, Hg * Dk: 2 * Hg * Dk], gp[:, 2 * Hg * Dk:]
    flop = N * Hg * (2.0 * Dk * Dv * 2 + 64 * (Dk + Dv))
    gbytes = N * Hg * (2 * Dk + 2 * Dv) * 2 + N * Hg * Dk * 4
    cases["gla_chunk 8 x 1024, 16 heads, 64 x 128"] = (
        lambda: M.gla(gq, gk, gv, dec, go, state, pre, q_scale=0.125, chunked=True), flop, gbytes)
    for parts in (4, 9):
        cases[f"gla_chunk 1 x 8192, {parts} spans"] = (
            lambda parts=parts: M.gla(gq, gk, gv, dec, go, state, long1, q_scale=0.125, chunked=True, parts=parts), flop, gbytes)
    Hs, P, S = 32, 64, 128
    xbc, dt, ys, ss = rn(N, Hs * P + 2 * S), rn(N, Hs), rn(N, Hs * P), rn(B, Hs, S, P, dtype=f32)
    vs = [torch.linspace(-3, 0, Hs, device=dev), torch.zeros(Hs, device=dev), torch.ones(Hs, device=dev)]
    sflop = N * Hs * (2.0 * S * P * 2 + 64 * (S + P))
    cases["like: ssd_chunk 8 x 1024, 32 heads, 128 x 64"] = (lambda: M.ssd(xbc, dt, ys, *vs, ss, 1, pre, chunked=True), sflop, N * Hs * P * 4)
    cases["like: ssd_chunk 1 x 8192, 4 spans"] = (
        lambda: M.ssd(xbc, dt, ys, *vs, ss, 1, long1, chunked=True, parts=4), sflop, N * Hs * P * 4)
    cases["gla_step decode 256"] = (lambda: M.gla(gq[:B], gk[:B], gv[:B], dec[:B], go[:B], state, one, q_scale=0.125), 0, B * Hg * Dk * Dv * 8)
    cases["like: ssd_step decode 256"] = (lambda: M.ssd(xbc[:B], dt[:B], ys[:B], *vs, ss, 1, one), 0, B * Hs * S * P * 8)
    a1, a2, ab = rn(N, 16), rn(Hg * Dk, 16, dtype=f32), rn(Hg * Dk, dtype=f32)
    cases["decay_gate 8192 x 1024, rank 16"] = (lambda: M.decay_gate(a1, a2, ab, 16.0), 0, N * Hg * Dk * 4)
    sa, st, so = rn(N, 128, dtype=f32), rn(VOCAB, 128), rn(N, 128)
    tok = torch.randint(0, VOCAB, (N,), device=dev, dtype=torch.int32)
    cases["like: token_side_gate 8192 x 128"] = (lambda: M.token_side_gate(sa, tok, st, 0, so, 128), 0, N * 128 * 8)
    # feed-forwards
    gu, act = rn(N, 8192), rn(N, 4096)
    cases["glu (gelu) 8192 x 4096"] = (lambda: M.glu(gu, act, M.Glu(1)), 0, N * 4096 * 6)
    cases["like: silu_mul 8192 x 4096"] = (lambda: M.silu_mul(gu, act), 0, N * 4096 * 6)
    wr = rn(E, W, s=0.02)
    cases["router logits 8192 x 32 x 2048"] = (lambda: K.gemm(h, wr, out_dtype=f32, deterministic=True), 0, N * W * 2)
    cases["gate_route 8192 x 4 of 32, rows to slots"] = (lambda: route(N, 256, h), 0, N * W * 2 * (1 + top))
    tables = torch.rand((VOCAB, E), device=dev, generator=gen).topk(top, -1).indices.to(torch.int32).contiguous()
    cases["like: table_route 8192 x 4, one layer"] = (lambda: X.table_route(tok, [(tables, E)], 256), 0, N * top * 12)
    cases["gate_route 64 x 4 of 32"] = (lambda: route(64, 1), 0, 64 * (E * 4 + top * 12))
    cases["like: table_route 64 x 4, one layer"] = (lambda: X.table_route(tok[:64], [(tables, E)], 1), 0, 64 * top * 12)
    up, down, wide = rn(E, 2 * ff, W, s=0.02), rn(E, W, ff, s=0.03), rn(2 * ff, W, s=0.02)
    mid, big, glu = rn(r256.max_slots, ff), rn(N * top, W), M.Glu(2, 7.0, 1.702, 1.0)
    eflop = 2.0 * N * top * W * ff
    cases["experts gate, up + clamped unit (grouped GEMM) 8192 x 4 of 32"] = (
        lambda: X.expert_product(by_slot, up, r256, gather=False, gate=glu), 2 * eflop, 0)
    cases["like: gemm 32768 x 2048 x 2048"] = (lambda: K.gemm(big, wide), 2 * eflop, 0)
    u1, m1 = rn(E, ff, W, s=0.02), rn(N * top, ff)
    cases["like: experts up + squared relu (grouped GEMM) 8192 x 4 of 32"] = (
        lambda: X.expert_product(by_slot, u1, r256, gather=False, act="relu2"), eflop, 0)
    cases["experts down (grouped GEMM) 8192 x 4 of 32"] = (lambda: X.expert_product(mid, down, r256, gather=False), eflop, 0)
    wd = rn(W, ff, s=0.03)
    cases["like: gemm 32768 x 2048 x 1024"] = (lambda: K.gemm(m1, wd), eflop, 0)
    r1, hd = route(64, 1)[0], rn(64, W)
    m64 = rn(r1.max_slots, ff)
    cases["experts gate, up + clamped unit (few rows) 64 x 4 of 32"] = (
        lambda: X.expert_product(hd, up, r1, gather=True, gate=glu), 0, E * 2 * ff * W * 2)
    cases["like: experts up + squared relu (few rows) 64 x 4 of 32"] = (
        lambda: X.expert_product(hd, u1, r1, gather=True, act="relu2"), 0, E * ff * W * 2)
    cases["experts down (few rows) 64 x 4 of 32"] = (lambda: X.expert_product(m64, down, r1, gather=False), 0, E * ff * W * 2)
    lg = rn(B, VOCAB, dtype=f32)
    cases["softcap, scaled 256 x 32000"] = (lambda: M.softcap_(lg, VOCAB, 30.0, 2.0), 0, B * VOCAB * 8)
    return cases


def kernel_lines(peaks: dict, only: str = "", iters: int = 20):
    from .kernels import _time
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    rows = []
    for name, (fn, flops, nbytes) in kernel_cases().items():
        if only and not re.search(only, name):
            continue
        ms, _ = _time(fn, iters, 3, flush)
        ideal = max(nbytes / (peaks["hbm_gbs"] * 1e9), flops / (peaks["bf16_tflops"] * 1e12)) * 1e3
        rows.append({"kernel": name, "us": ms * 1e3, "roofline_us": ideal * 1e3, "fraction": ideal / ms})
    return rows


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="1024,2048,4096")
    ap.add_argument("--kernels", action="store_true")
    ap.add_argument("--peaks", default="MEASURED_PEAKS.json")
    ap.add_argument("--only", default="")
    ap.add_argument("--iters", type=int, default=10)
    args = ap.parse_args(argv)
    try:
        with open(args.peaks) as f:
            peaks = json.load(f)
    except OSError:
        peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    if args.kernels:
        for r in kernel_lines(peaks, args.only):
            print(f"{r['kernel']:78s} {r['us']:9.1f} us  roofline {r['roofline_us']:8.1f} us  {r['fraction']:.3f} of measured")
        return 0
    for r in model_lines([int(s) for s in args.sizes.split(",")], args.iters):
        print(json.dumps(r))
    return 0


if __name__ == "__main__":
    sys.exit(main())
