"""Serving speed of a Gugedra model beside a GPT-2 model of the same width and depth, and the roofline of its kernels.

    python -m nexus_b200.bench.hybrid [--sizes 1024,2048,4096] [--kernels] [--peaks MEASURED_PEAKS.json] [--only REGEX]

Model lines (random weights, BF16): prefill = tokens / s of one packed step of fresh prompts, CUDA-event time, median over
steps; decode = tokens / s of one-token steps of a batch of sequences with 1024 tokens behind them (captured graphs).  The
weights of both models exceed the L2 cache, so it needs no flush between steps.

Kernel lines (``--kernels``): every kernel of the design at the sizes of the 2048-wide model, cold L2, as a fraction of the
roofline time max(bytes / measured copy bandwidth, FLOPs / measured BF16 rate), beside the like kernels of the GPT-2 engine.
"""
from __future__ import annotations

import argparse
import json
import re
import statistics
import sys

import torch

# width, layers, attention head size; GPT-2: width / head size heads and a 4 x feed-forward
SIZES = {1024: (12, 64), 2048: (12, 64), 4096: (6, 128)}
VOCAB = 32000


def hybrid_config(width: int, layers: int, dim: int):
    """Two parallel layers, then a delta layer, and so on; window 1024, 4 query heads to a KV head, SSD inner = width with
    128 state rows, feed-forward of 2.75 x width."""
    from ..lm.hybrid import AttentionSpec, DeltaSpec, HybridConfig, HybridLayer, ParallelSpec, SsdSpec
    heads = width // dim
    par = ParallelSpec(AttentionSpec(heads, heads // 4, dim, dim, dim ** -0.5, 30.0, 1024, dim // 2, 250000.0),
                       SsdSpec(width // 64, 64, 128, 1, 4, 1), 0.8, 1.1)
    delta = DeltaSpec(width // 128, width // 256, 128, 128, 4)
    ff = width * 11 // 4
    out = [HybridLayer(delta, ff) if i % 3 == 2 else HybridLayer(par, ff) for i in range(layers)]
    return HybridConfig(VOCAB, width, out, 1e-6, 128, 15.0, f"gugedra-{width}")


def _step_ms(fn, iters: int, warm: int = 3) -> float:
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    out = []
    for _ in range(iters):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        b.synchronize()
        out.append(a.elapsed_time(b))
    return statistics.median(out)


def time_engine(weights, prompts=(8, 1024), long_prompt=4096, batch=64, iters=10) -> dict:
    """Prefill of ``prompts`` (count, length), of one long prompt, and decode of ``batch`` sequences."""
    from ..infer import Chunk, EngineConfig, create_engine
    from ..ops import _cuda as K
    ctx = max(long_prompt, 1024 + 64) + 64
    eng = create_engine(weights, EngineConfig(max_seqs=batch, max_tokens=8192, kv_tokens=batch * 1280 + 8192, context=ctx))
    g = torch.Generator().manual_seed(0)
    V = eng.vocab()

    def toks(n):
        return torch.randint(0, V, (n,), generator=g).tolist()

    def prefill(count, length):
        batch_tokens = [toks(length) for _ in range(count)]

        def run():
            ids = [eng.add_sequence() for _ in range(count)]
            eng.forward([Chunk(s, t, 1) for s, t in zip(ids, batch_tokens)])
            for s in ids:
                eng.free_sequence(s)
        return count * length / (_step_ms(run, iters) * 1e-3)
    out = {"prefill_tok_s": prefill(*prompts), "prefill_long_tok_s": prefill(1, long_prompt)}
    ids = [eng.add_sequence() for _ in range(batch)]
    for i in range(0, batch, 8):
        eng.forward([Chunk(s, toks(1024), 0) for s in ids[i: i + 8]])
    one = toks(batch)
    ms = _step_ms(lambda: eng.forward([Chunk(s, [t], 1, True) for s, t in zip(ids, one)]), 30)
    out["decode_tok_s"], out["decode_ms"] = batch / (ms * 1e-3), ms
    K.check_status()
    out["parameters"] = weights.parameters()
    del eng
    torch.cuda.empty_cache()
    return out


def model_lines(sizes, iters=10):
    from ..infer import Gpt2Weights
    from ..lm.hybrid import random_gugedra
    rows = []
    for width in sizes:
        layers, dim = SIZES[width]
        hy = time_engine(random_gugedra(hybrid_config(width, layers, dim)), iters=iters)
        gp = time_engine(Gpt2Weights.random(layers, width // dim, width, VOCAB, 4096 + 64), iters=iters)
        rows.append({"width": width, "layers": layers, "gugedra": hy, "gpt2": gp})
    return rows


# ------------------------------------------------------------------------------------------ kernels
def kernel_cases():
    """name -> (launch, flops, bytes)."""
    from ..ops import _cuda as K
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
    W, N, B, cases = 2048, 8192, 256, {}
    pre, one, long1 = segs([1024] * 8, 0), segs([1] * B, 1023), segs([N], 0)
    ones = torch.ones(W, device=dev)
    x, y, h = rn(N, W, dtype=torch.float32), rn(N, W), rn(N, W)
    cases["residual_norm (post-norm, add, next norm) 8192x2048"] = (
        lambda: M.residual_norm(x, y=y, w_post=ones, w_next=ones, h=h, eps=1e-6), 0, N * W * (4 + 2 + 4 + 2))
    xb = rn(N, W, dtype=torch.float32)
    cases["like: layernorm fp32 -> bf16 8192x2048"] = (
        lambda: K.norm_fwd(xb, ones, ones, out_dtype=bf, want_stats=False), 0, N * W * 6)
    # attention: 32 query heads, 8 KV heads, D 64, window 1024
    H, G, D, win, bs = 32, 8, 64, 1024, 16
    blocks = B * 1024 // bs
    kc, vc = rn(blocks, bs, G, D), rn(blocks, bs, G, D)
    table = torch.randperm(blocks, generator=torch.Generator().manual_seed(1)).view(B, -1).to(torch.int32).to(dev)
    proj = rn(N, (H + 2 * G) * D)
    pos = (torch.arange(N, dtype=torch.int32) % 1024).to(dev)
    slot = torch.arange(N, dtype=torch.int32, device=dev)
    cos, sin = rn(1024, 16, dtype=torch.float32), rn(1024, 16, dtype=torch.float32)
    cases["rope_append 8192 x (32+8+8) x 64"] = (
        lambda: M.rope_append(proj, 0, H * D, (H + G) * D, H, G, D, D, 32, pos, slot, cos, sin, kc, vc), 0,
        N * (H * 32 * 4 + G * D * 2 * 4 + G * 32 * 2))
    kg, vg = rn(N, G, D), rn(N, G, D)
    cases["like: rope 8192 x 32 x 64 (all dims)"] = (lambda: I.rope_(proj[:, : H * D].view(N, H, D), pos, rn_cos, rn_sin), 0,
                                                     N * H * D * 4)
    rn_cos, rn_sin = rn(1024, 32, dtype=torch.float32), rn(1024, 32, dtype=torch.float32)
    cases["like: kv_append 8192 x 8 x 64"] = (lambda: I.kv_append(kg, vg, slot, kc, vc), 0, N * G * D * 8)
    out = rn(N, H * D)
    kw = dict(heads=H, block_size=bs, window=win, scale=0.125, softcap=30.0)
    pairs8 = 8 * 1024 * 1025 // 2
    cases["paged_window_prefill (mma) 8 x 1024, window 1024"] = (
        lambda: M.paged_window_attention(proj[:, : H * D], kc, vc, table, out, pre, **kw), 4.0 * D * H * pairs8, 0)
    q4, k4, v4 = rn(8, 1024, H, D), rn(8, 1024, G, D), rn(8, 1024, G, D)
    cases["flash soft-capped 8 x 1024"] = (lambda: K.attention_fwd(q4, k4, v4, window=win, softcap=30.0), 4.0 * D * H * pairs8, 0)
    cases["like: flash plain 8 x 1024"] = (lambda: K.attention_fwd(q4, k4, v4), 4.0 * D * H * pairs8, 0)
    qd, od = rn(B, H * D), rn(B, H * D)
    cases["paged_window_decode 256 x 1024, 32 / 8 heads"] = (
        lambda: M.paged_window_attention(qd, kc, vc, table, od, one, **kw), 0, B * 1024 * G * D * 4)
    Hg = 8
    qg, og = rn(B, Hg, D), rn(B, Hg, D)
    rows, ctx = torch.arange(B, dtype=torch.int32, device=dev), torch.full((B,), 1024, dtype=torch.int32, device=dev)
    cases["like: paged_decode (TMA) 256 x 1024, 8 / 8 heads"] = (
        lambda: I.paged_attention(qg, kc, vc, table, rows, ctx, og, block_size=bs, kv_heads=G), 0, B * 1024 * G * D * 4)
    # state space: 32 heads of 64, state 128, one group
    Hs, P, S = 32, 64, 128
    C = Hs * P + 2 * S
    xin, xbc, w, b = rn(N, C), rn(N, C), rn(4, C, dtype=torch.float32), rn(C, dtype=torch.float32)
    tail = rn(B, 3, C)
    cases["conv_silu 8192 x 2304, 4 taps"] = (lambda: M.conv_silu(xin, xbc, w, b, tail, pre), 0, N * C * 4)
    cases["conv_silu decode 256 x 2304"] = (lambda: M.conv_silu(xin[:B], xbc[:B], w, b, tail, one), 0, B * C * 2 * 8)
    dt, ys, state = rn(N, Hs), rn(N, Hs * P), rn(B, Hs, S, P, dtype=torch.float32)
    v = [torch.linspace(-3, 0, Hs, device=dev), torch.zeros(Hs, device=dev), torch.ones(Hs, device=dev)]
    flop = N * Hs * (2.0 * S * P * 2 + 64 * (S + P))
    cases["ssd_chunk 8 x 1024"] = (lambda: M.ssd(xbc, dt, ys, *v, state, 1, pre, chunked=True), flop, N * Hs * P * 4)
    for parts in (2, 4, 9):
        cases[f"ssd_chunk 1 x 8192, {parts} spans"] = (
            lambda parts=parts: M.ssd(xbc, dt, ys, *v, state, 1, long1, chunked=True, parts=parts), flop, N * Hs * P * 4)
    cases["ssd_step decode 256"] = (lambda: M.ssd(xbc[:B], dt[:B], ys[:B], *v, state, 1, one), 0, B * Hs * S * P * 8)
    z, wn, zo = rn(N, Hs * P), rn(Hs * P, dtype=torch.float32), rn(N, Hs * P)
    cases["gated_norm 8192x2048, one group"] = (
        lambda: M.gated_norm(ys, z, wn, zo, groups=1, gate_first=True, eps=1e-6), 0, N * Hs * P * 6)
    # delta rule: 16 value heads, 8 key heads, 128 x 128
    Hd, Gd, Dd = 16, 8, 128
    Cd = (2 * Gd + Hd) * Dd
    qkv, ba, o = rn(N, Cd), rn(N, 2 * Hd), rn(N, Hd * Dd)
    sd = rn(B, Hd, Dd, Dd, dtype=torch.float32)
    dv = [torch.linspace(-4, -1, Hd, device=dev), torch.zeros(Hd, device=dev)]
    dk = dict(unit_eps=1e-6, q_scale=Dd ** -0.5)
    dflop = N * Hd * (6.0 * Dd * Dd + 64 * (2 * Dd + 2 * Dd) + 64 * 64)
    for name, sg in (("8 x 1024", pre), ("1 x 8192", long1)):
        cases[f"delta prep + chunk {name}"] = (
            lambda sg=sg: M.delta(qkv, ba[:, :Hd], ba[:, Hd:], o, *dv, sd, Gd, sg, chunked=True, **dk), dflop, N * (Cd + Hd * Dd) * 2)
    cases["delta_step decode 256"] = (
        lambda: M.delta(qkv[:B], ba[:B, :Hd], ba[:B, Hd:], o[:B], *dv, sd, Gd, one, **dk), 0, B * Hd * Dd * Dd * 8)
    wd, go = torch.ones(Dd, device=dev), rn(N, Hd * Dd)
    cases["gated_norm 8192 x 16 x 128 per head"] = (
        lambda: M.gated_norm(o, z[:, : Hd * Dd], wd, go, groups=Hd, gate_first=False, eps=1e-6), 0, N * Hd * Dd * 6)
    F = 5632
    gu, act = rn(N, 2 * F), rn(N, F)
    cases["silu_mul 8192 x 5632"] = (lambda: M.silu_mul(gu, act), 0, N * F * 6)
    cases["like: gated_fwd 8192 x 5632"] = (lambda: I.gated_fwd(gu), 0, N * F * 6)
    sa, st, so = rn(N, 128, dtype=torch.float32), rn(VOCAB, 128 * 12), rn(N, 128)
    tok = torch.randint(0, VOCAB, (N,), device=dev, dtype=torch.int32)
    cases["token_side_gate 8192 x 128"] = (lambda: M.token_side_gate(sa, tok, st, 256, so, 128), 0, N * 128 * 8)
    lg = rn(B, VOCAB, dtype=torch.float32)
    cases["softcap 256 x 32000"] = (lambda: M.softcap_(lg, VOCAB, 15.0), 0, B * VOCAB * 8)
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
            print(f"{r['kernel']:58s} {r['us']:9.1f} us  roofline {r['roofline_us']:8.1f} us  {r['fraction']:.3f} of measured")
        return 0
    for r in model_lines([int(s) for s in args.sizes.split(",")], args.iters):
        print(json.dumps(r))
    return 0


if __name__ == "__main__":
    sys.exit(main())
