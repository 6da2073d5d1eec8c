"""Serving speed of a Makuzen model beside the framework's other models of the same width and depth, and the roofline of its
kernels.

    python -m nexus_b200.bench.latent [--sizes 1024,2048,4096] [--kernels] [--peaks MEASURED_PEAKS.json] [--only REGEX]

The measurements are those of `bench.hybrid` (packed prefill of fresh prompts, captured decode steps of 64 sequences with
1024 tokens behind them, kernels with a cold L2 against the measured peaks)."""
from __future__ import annotations

import argparse
import json
import re
import sys

import torch

from .hybrid import SIZES, VOCAB, hybrid_config, time_engine


def latent_config(width: int, layers: int):
    """Heads of 128 + 64 with a latent of 512, window 1024, 32 experts of width / 2 of which a token uses 4, a shared expert of
    the model's width."""
    from ..lm.config import RopeScaling
    from ..lm.hybrid import ExpertsSpec, HybridConfig, HybridLayer, LatentSpec
    mix = LatentSpec(width // 128, 128, 64, 128, width * 3 // 8, 512, 192 ** -0.5, 1024, 250000.0, RopeScaling("yarn", 4.0, 4096))
    out = [HybridLayer(mix, experts=ExpertsSpec(32, 4, width // 2, width)) for _ in range(layers)]
    return HybridConfig(VOCAB, width, out, 1e-5, name=f"makuzen-{width}", pre_norm=False, embed_scale=2.0, residual_mult=0.4)


def active_parameters(cfg) -> int:
    """Weights one token meets (embedding row aside)."""
    n = cfg.vocab * cfg.width
    for layer in cfg.layers:
        m, f = layer.mixer, layer.experts
        n += cfg.width * (m.q_rank + m.kv_rank + m.rope_dims + m.heads * (m.vdim + 1)) + m.q_rank * m.heads * (m.dim + m.rope_dims)
        n += m.kv_rank * m.heads * (m.dim + m.vdim) + 2 * cfg.width * (f.top * f.ff + f.shared)
    return n


def model_lines(sizes, iters=10):
    from ..infer import Gpt2Weights
    from ..lm.hybrid import random_gugedra
    from ..lm.makuzen import random_makuzen
    rows = []
    for width in sizes:
        layers, dim = SIZES[width]
        cfg = latent_config(width, layers)
        mk = time_engine(random_makuzen(cfg), iters=iters)
        mk["active_parameters"] = active_parameters(cfg)
        gu = time_engine(random_gugedra(hybrid_config(width, layers, dim)), iters=iters)
        gp = time_engine(Gpt2Weights.random(layers, width // dim, width, VOCAB, 4096 + 64), iters=iters)
        rows.append({"width": width, "layers": layers, "makuzen": mk, "gugedra": gu, "gpt2": gp})
    return rows


# ------------------------------------------------------------------------------------------ kernels
def kernel_cases():
    """name -> (launch, flops, bytes)."""
    from ..ops import _cuda as K
    from ..ops import _experts as X
    from ..ops import _infer as I
    from ..ops import _mixers as M
    dev, bf = "cuda", torch.bfloat16
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
    W, N, H, D, R, Dv, rank, q_rank, bs, cases = 2048, 8192, 16, 128, 64, 128, 512, 768, 16, {}
    row, head = rank + R, D + R
    ones, x, y, h = torch.ones(W, device=dev), rn(N, W, dtype=torch.float32), rn(N, W), rn(N, W)
    E, top, ff = 32, 4, 1024
    tokens = torch.randint(0, VOCAB, (N,), device=dev, dtype=torch.int32)
    tables = [torch.rand((VOCAB, E), device=dev, generator=gen).topk(top, -1).indices.to(torch.int32).contiguous() for _ in range(12)]

    def route(n, align):
        return X.table_route(tokens[:n], [(tables[0], E)], align)[0]
    r256 = route(N, 256)
    by_slot = rn(r256.max_slots, W)
    gate, dot = rn(N, dtype=torch.float32), torch.empty(N, device=dev)
    cases["residual_norm + gate of the shared expert + rows to expert slots 8192x2048"] = (
        lambda: M.residual_norm(x, y=y, w_post=ones, x_cast=h, eps=1e-5, w_dot=ones, dot_out=dot, scatter=by_slot, slots=r256.slots,
                                top=top), 0, N * W * (4 + 2 + 4 + 2 + 2 * top))
    cases["residual_norm + sum of 4 experts and the shared one 8192x2048"] = (
        lambda: M.residual_norm(x, y=y, w_post=ones, x_cast=h, eps=1e-5, experts=by_slot, slots=r256.slots, top=top, y_gate=gate), 0,
        N * W * (4 + 2 + 4 + 2 + 2 * top))
    cases["like: residual_norm 8192x2048"] = (lambda: M.residual_norm(x, y=y, w_post=ones, w_next=ones, h=h, eps=1e-6), 0, N * W * 12)
    cases["like: layernorm fp32 -> bf16 8192x2048"] = (
        lambda: K.norm_fwd(x, ones, ones, out_dtype=bf, want_stats=False), 0, N * W * 6)
    # latent attention
    B, ctx = 256, 1024
    cache = rn(B * ctx // bs, bs, 1, row)
    table = torch.randperm(B * ctx // bs, generator=torch.Generator().manual_seed(1)).view(B, -1).to(torch.int32).to(dev)
    proj = rn(N, q_rank + rank + R + H)
    pos, slot = (torch.arange(N, dtype=torch.int32) % 1024).to(dev), torch.arange(N, dtype=torch.int32, device=dev)
    cos, sin = rn(1024, R // 2, dtype=torch.float32), rn(1024, R // 2, dtype=torch.float32)
    cq, lat, hg, q = rn(N, q_rank), rn(N, row), torch.rand((N, H), device=dev), rn(N, H * head)
    wq, wk = torch.ones(q_rank, device=dev), torch.ones(rank, device=dev)
    off = (0, q_rank, q_rank + rank, q_rank + row)
    cases["latent_prep 8192 x (768 + 512 + 64 + 16)"] = (
        lambda: M.latent_prep(proj, off, q_rank, rank, R, H, wq, wk, pos, slot, cos, sin, cq, cache, rank, hg, eps=1e-5, lat=lat), 0,
        N * 2 * (2 * q_rank + 3 * row + H) + N * H * 4)
    cases["rope_heads 8192 x 16 x 64 of 192"] = (
        lambda: M.rope_heads(q, head, D, q, head, D, H, R, R, pos, cos, sin), 0, N * H * R * 4)
    kc, vc = rn(B * ctx // bs, bs, 8, 64), rn(B * ctx // bs, bs, 8, 64)
    pr = rn(N, 48 * 64)
    cos32, sin32 = rn(1024, 16, dtype=torch.float32), rn(1024, 16, dtype=torch.float32)
    cases["like: rope_append 8192 x (32+8+8) x 64"] = (
        lambda: M.rope_append(pr, 0, 2048, 2560, 32, 8, 64, 64, 32, pos, slot, cos32, sin32, kc, vc), 0,
        N * (32 * 32 * 4 + 8 * 64 * 2 * 4 + 8 * 32 * 2))
    kv, out = rn(N, H * (D + Dv)), rn(N, H * Dv)

    def blocks(count, length, window):
        back = window - 1 if window else 1 << 30
        b = [(min(p, back) + 256, i * length + p, 256, p, i * length) for i in range(count) for p in range(0, length, 256)]
        b.sort(key=lambda t: -t[0])
        return torch.tensor([t[1:] for t in b], dtype=torch.int32, device=dev)

    def pairs(count, length, window):
        return count * sum(min(i + 1, window) if window else i + 1 for i in range(length))
    for count, length, window in ((8, 1024, 0), (2, 4096, 0), (2, 4096, 1024)):
        bl = blocks(count, length, window)
        cases[f"latent_prompt {count} x {length}" + (f", window {window}" if window else "")] = (
            lambda bl=bl, window=window: M.latent_prompt(q, kv, lat, out, bl, heads=H, dim=D, rot=R, vdim=Dv, rank=rank, window=window,
                                                         scale=0.07, gate=hg), 2.0 * (D + R + Dv) * H * pairs(count, length, window), 0)
        q4, k4, v4 = (rn(count, length, H, 128) for _ in range(3))
        cases[f"like: flash, head size 128, {count} x {length}" + (f", window {window}" if window else "")] = (
            lambda q4=q4, k4=k4, v4=v4, window=window: K.attention_fwd(q4, k4, v4, window=window), 4.0 * 128 * H * pairs(count, length, window), 0)
    runs = torch.tensor([[i * 1024, 1024, 0, i] for i in range(8)], dtype=torch.int32, device=dev)
    cases["latent_gather 8 x 1024 rows of 576"] = (lambda: M.latent_gather(cache, table, runs, 1024, lat), 0, N * row * 4)
    one = segs([1] * B, ctx - 1)
    for heads in (16, 32):
        ql, ol, g1 = rn(B, heads * row), rn(B, heads * rank), torch.rand((B, heads), device=dev)
        cases[f"latent_attention, decode 256 x 1024, {heads} heads"] = (
            lambda ql=ql, ol=ol, g1=g1, heads=heads: M.latent_attention(ql, cache, table, ol, one, heads=heads, rank=rank, window=1024,
                                                                        scale=0.07, gate=g1), 0, B * ctx * row * 2)
    qd, od = rn(B, 32 * 64), rn(B, 32 * 64)
    cases["like: paged_window_decode 256 x 1024, 32 / 8 heads"] = (
        lambda: M.paged_window_attention(qd, kc, vc, table, od, one, heads=32, block_size=bs, window=1024, scale=0.125), 0,
        B * ctx * 8 * 64 * 4)
    short = segs([8] * 32, ctx - 8)
    qs, os_, gs = rn(B, H * row), rn(B, H * rank), torch.rand((B, H), device=dev)
    cases["latent_attention, 32 portions of 8 behind 1016"] = (
        lambda: M.latent_attention(qs, cache, table, os_, short, heads=H, rank=rank, window=1024, scale=0.07, gate=gs, splits=2),
        2.0 * B * H * ctx * (row + rank), 32 * ctx * row * 2)
    pq, po = rn(B, 32 * 64), rn(B, 32 * 64)
    cases["like: paged_window_prefill, 32 portions of 8 behind 1016, 32 / 8 heads"] = (
        lambda: M.paged_window_attention(pq, kc, vc, table, po, short, heads=32, block_size=bs, window=1024, scale=0.125),
        4.0 * B * 32 * 64 * ctx, 32 * ctx * 8 * 64 * 4)
    uk, uv, qn, ql = rn(H, rank, D), rn(H, Dv, rank), rn(64, H, head), rn(64, H, row)
    on, av = rn(64, H, rank), rn(64, H, Dv)
    cases["W_uk on the query side, 64 rows x 16 heads"] = (
        lambda: X.head_product(qn[:, :, :D], uk, ql[:, :, :rank]), 0, H * D * rank * 2 + 64 * H * (D + rank) * 2)
    cases["W_uv on the weighted latents, 64 rows x 16 heads"] = (
        lambda: X.head_product(on, uv, av), 0, H * Dv * rank * 2 + 64 * H * (Dv + rank) * 2)
    sw = rn(4096, 512, s=0.05)
    xs = rn(64, 512)
    cases["like: gemm 64 x 4096 x 512 (split K)"] = (lambda: K.gemm(xs, sw, split_k=0, block_n=128, deterministic=True), 0, 4096 * 512 * 2)
    # experts
    up, down = rn(E, ff, W, s=0.02), rn(E, W, ff, s=0.03)
    mid = rn(r256.max_slots, ff)
    flop = 2.0 * N * top * W * ff
    cases["experts up (grouped GEMM, squared relu) 8192 x 4 of 32"] = (
        lambda: X.expert_product(by_slot, up, r256, gather=False, act="relu2"), flop, 0)
    cases["experts down (grouped GEMM) 8192 x 4 of 32"] = (lambda: X.expert_product(mid, down, r256, gather=False), flop, 0)
    big, wu, wd, mid2 = rn(N * top, W), rn(ff, W), rn(W, ff), rn(N * top, ff)
    cases["like: gemm 32768 x 1024 x 2048"] = (lambda: K.gemm(big, wu), flop, 0)
    cases["like: gemm 32768 x 2048 x 1024"] = (lambda: K.gemm(mid2, wd), flop, 0)
    r1, hd = route(64, 1), rn(64, W)
    m1 = rn(r1.max_slots, ff)
    cases["experts up (few rows) 64 x 4 of 32"] = (
        lambda: X.expert_product(hd, up, r1, gather=True, act="relu2"), 0, E * ff * W * 2)
    cases["experts down (few rows) 64 x 4 of 32"] = (lambda: X.expert_product(m1, down, r1, gather=False), 0, E * ff * W * 2)
    wide = rn(E * ff // 2, W, s=0.02)
    cases["like: gemm 64 x 16384 x 2048 (split K)"] = (lambda: K.gemm(hd, wide, split_k=0, block_n=128, deterministic=True), 0,
                                                      E * ff // 2 * W * 2)
    cases["table_route 8192 x 4, 12 layers"] = (lambda: X.table_route(tokens, [(t, E) for t in tables], 256), 0, N * top * 12 * 12)
    gu = rn(N, 2 * W)
    cases["like: gated_fwd 8192 x 2048"] = (lambda: I.gated_fwd(gu), 0, N * W * 6)
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
