"""Serving speed of a Lukopel model beside the framework's other models of the same width and depth, and the roofline of its
kernels.

    python -m nexus_b200.bench.talking [--sizes 1024,2048,4096] [--kernels] [--peaks MEASURED_PEAKS.json] [--only REGEX]

The measurements are those of `bench.hybrid` (packed prefill of fresh prompts, captured decode steps of 64 sequences with
1024 tokens behind them, kernels with a cold L2 against the measured peaks)."""
from __future__ import annotations

import argparse
import json
import re
import sys

import torch

from .hybrid import SIZES, VOCAB, time_engine


def talking_config(width: int, runs: int, dim: int):
    """Attention in chunks of 1024 and attention with heads that mix in turn, 4 query heads to a KV head, 128 bias distances; a
    squared-relu feed-forward of 4 x width; 4 residual streams.  ``runs`` layers run: two of them are run twice."""
    from ..lm.hybrid import DistanceBias, HybridConfig, HybridLayer, Loop, NormedAttentionSpec, QueryTemperature
    heads = width // dim
    chunked = NormedAttentionSpec(heads, heads // 4, dim, dim, dim ** -0.5, norm="all", bias=True, head_scale=True, chunk=1024)
    talking = NormedAttentionSpec(heads, heads // 4, dim, dim, dim ** -0.5, unit_values=True, temperature=QueryTemperature(0.1, 512),
                                  distance=DistanceBias(32, 128), talk=True, gate=True)
    out = [HybridLayer((chunked, talking)[i % 2], ff=4 * width, act="relu2", ff_bias=True) for i in range(runs - 2)]
    return HybridConfig(VOCAB, width, out, 1e-5, name=f"lukopel-{width}", post_norm=False, streams=4, loop=Loop(0, 2, 2), positions=8192)


def model_lines(sizes, iters=10):
    from ..infer import Gpt2Weights
    from ..lm.gutivik import random_gutivik
    from ..lm.lukopel import random_lukopel
    from .routed import active_parameters, routed_config
    rows = []
    for width in sizes:
        layers, dim = SIZES[width]
        lk = time_engine(random_lukopel(talking_config(width, layers, dim)), iters=iters)
        routed = routed_config(width, layers, dim)
        gt = time_engine(random_gutivik(routed), iters=iters)
        gt["active_parameters"] = active_parameters(routed)
        gp = time_engine(Gpt2Weights.random(layers, width // dim, width, VOCAB, 4096 + 64), iters=iters)
        rows.append({"width": width, "layer_runs": layers, "lukopel": lk, "gutivik": gt, "gpt2": gp})
    return rows


# ------------------------------------------------------------------------------------------ kernels
def kernel_cases():
    """name -> (launch, flops, bytes)."""
    from ..infer.prompt import row_slices
    from ..ops import _cuda as K
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
    W, N, B, bs, S, cases = 2048, 8192, 256, 16, 4, {}
    one, short = segs([1] * B, 1023), segs([8] * 32, 1016)
    ones, x, y, h = torch.ones(W, device=dev), rn(N, S, W, dtype=f32), rn(N, W), rn(N, W)
    mix, vec = torch.eye(S, device=dev) * 0.8 + 0.05, torch.ones(S, device=dev)
    for n in (N, 64):
        step = dict(y=y[:n], mix=mix, out=vec, read=vec * 0.25, w_next=ones, h=h[:n], eps=1e-5)
        cases[f"stream_residual (4 streams, next norm) {n}x2048"] = (
            lambda n=n, step=step: M.stream_residual(x[:n], **step), 0, n * W * (S * 8 + 4))
        x1 = rn(n, W, dtype=f32)
        cases[f"like: residual_norm (add, next norm) {n}x2048"] = (
            lambda n=n, x1=x1: M.residual_norm(x1, y=y[:n], w_next=ones, h=h[:n], eps=1e-5), 0, n * W * 12)
    pos, slot = (torch.arange(N, dtype=torch.int32) % 1024).to(dev), torch.arange(N, dtype=torch.int32, device=dev)

    def blocks(count, length, window):
        back = window - 1 if window else 1 << 30
        b = [(min(p, back) + 256, i * length + p, 256, p, i * length) for i in range(count) for p in range(0, length, 256)]
        b.sort(key=lambda t: -t[0])
        return torch.tensor([t[1:] for t in b], dtype=torch.int32, device=dev)

    def pairs(count, length, chunk=0):
        return count * sum(i % chunk + 1 if chunk else i + 1 for i in range(length))
    for H, G, D in ((32, 8, 64), (32, 8, 128)):
        sizes = f"{H} / {G} heads of {D}"
        kc, vc = rn(B * 1024 // bs, bs, G, D), rn(B * 1024 // bs, bs, G, D)
        table = torch.randperm(B * 1024 // bs, generator=torch.Generator().manual_seed(1)).view(B, -1).to(torch.int32).to(dev)
        q0, k0, v0, g0 = 0, H * D, (H + G) * D, (H + 2 * G) * D
        proj, gate = rn(N, g0 + 64), torch.rand((N, H), device=dev)
        wq, wk = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev)
        prep = dict(heads=H, kv_heads=G, dim=D, vdim=D, norm_dim=D, norm_vdim=D, eps=1e-5, w_q=wq, w_k=wk, positions=pos, slots=slot,
                    k_cache=kc, v_cache=vc, q_scale=D ** -0.5, store_kv=True)
        nbytes = (H + G) * D * 4 + 2 * G * D * 2 + G * D * 4
        for n in (N, B):
            cases[f"head_prep (per head, unit values, gate) {n} x {sizes}"] = (
                lambda n=n, prep=prep, proj=proj, gate=gate: M.head_prep(proj[:n], (q0, k0, v0, g0), unit_values=True, coef=0.1, every=512,
                                                                         gate=gate[:n], **prep), 0, n * (nbytes + H * 6))
            cases[f"head_prep (whole projection) {n} x {sizes}"] = (
                lambda n=n, prep=prep, proj=proj: M.head_prep(proj[:n], (q0, k0, v0, g0), norm_all=True, **prep), 0, n * (nbytes - G * D * 2))
            cos, sin = rn(1024, D // 4, dtype=f32), rn(1024, D // 4, dtype=f32)
            cases[f"like: rope_append {n} x {sizes}"] = (
                lambda n=n, proj=proj, kc=kc, vc=vc, cos=cos, sin=sin, D=D, H=H, G=G, k0=k0, v0=v0: M.rope_append(
                    proj[:n], 0, k0, v0, H, G, D, D, D // 2, pos, slot, cos, sin, kc, vc), 0,
                n * (H * D // 2 * 4 + G * D * 2 * 4 + G * D // 2 * 2))
        rel, talk = rn(H, 129, dtype=f32), torch.eye(H, device=dev) * 0.8 + rn(H, H, dtype=f32, s=0.1)
        ext = M.extended_bias(rel)
        qkv = rn(N, g0 + 64)
        qkv[:, : H * D] *= D ** -0.5            # as normed queries that carry the scale of the scores
        q, k, v = qkv[:, : H * D], qkv[:, k0: v0], qkv[:, v0: g0]
        out, wide = rn(N, H * D), rn(N, H * G * D)
        kw = dict(heads=H, kv_heads=G, dim=D, vdim=D, scale=1.0)
        for count, length in ((8, 1024), (2, 4096)):
            bl, p = blocks(count, length, 0), pairs(count, length)
            mixing = 2.0 * H * H * p
            slices = [(torch.tensor(g, dtype=torch.int32, device=dev), r, n) for g, r, n in row_slices(bl.tolist(), M.talk_rows(H, G, D))]
            cases[f"prompt attention, heads that mix, {count} x {length}, {sizes}"] = (
                lambda slices=slices, q=q, k=k, v=v, out=out, ext=ext, talk=talk, gate=gate, kw=kw: M.talk_prompt_mixed(
                    q, k, v, out, slices, talk, gate, window=0, bias=ext, distances=129, **kw), 4.0 * D * H * p + mixing, 0)
            cases[f"prompt attention with distance biases, {count} x {length}, {sizes}"] = (
                lambda bl=bl, q=q, k=k, v=v, out=out, rel=rel, kw=kw: M.window_prompt(q, k, v, out, bl, window=0, bias=rel, **kw),
                4.0 * D * H * p, 0)
            cases[f"prompt attention in chunks of 1024, {count} x {length}, {sizes}"] = (
                lambda bl=bl, q=q, k=k, v=v, out=out, kw=kw: M.window_prompt(q, k, v, out, bl, window=0, chunk=1024, **kw),
                4.0 * D * H * pairs(count, length, 1024), 0)
            cases[f"like: window_prompt, window 1024, {count} x {length}, {sizes}"] = (
                lambda bl=blocks(count, length, 1024), q=q, k=k, v=v, out=out, kw=kw: M.window_prompt(q, k, v, out, bl, window=1024, **kw),
                4.0 * D * H * count * sum(min(i + 1, 1024) for i in range(length)), 0)
            q4, k4, v4 = rn(count, length, H, D), rn(count, length, G, D), rn(count, length, G, D)
            cases[f"like: flash {count} x {length}, {sizes}"] = (
                lambda q4=q4, k4=k4, v4=v4: K.attention_fwd(q4, k4, v4), 4.0 * D * H * p, 0)
        cases[f"head_mix {N} x {sizes}"] = (
            lambda wide=wide, out=out, talk=talk, gate=gate, H=H, G=G, D=D: M.head_mix(wide, talk, gate, out, heads=H, kv_heads=G, vdim=D),
            0, N * H * D * 2 * (G + 1))
        pk = dict(heads=H, block_size=bs, window=0, scale=1.0)
        qd, od = q[:B], out[:B]
        kv = B * 1024 * G * D * 4
        cases[f"talk_paged, decode 256 x 1024, {sizes}"] = (
            lambda qd=qd, od=od, kc=kc, vc=vc, table=table, rel=rel, talk=talk, gate=gate, pk=pk: M.talk_paged(
                qd, kc, vc, table, od, talk, one, keys=1024, gate=gate, bias=rel, **pk), 0, kv)
        cases[f"paged decode in chunks of 1024, 256 x 1024, {sizes}"] = (
            lambda qd=qd, od=od, kc=kc, vc=vc, table=table, pk=pk: M.paged_window_attention(qd, kc, vc, table, od, one, chunk=1024, **pk), 0, kv)
        cases[f"like: paged_window_decode 256 x 1024, {sizes}"] = (
            lambda qd=qd, od=od, kc=kc, vc=vc, table=table, pk=pk: M.paged_window_attention(qd, kc, vc, table, od, one, **pk), 0, kv)
        cases[f"talk_paged, 32 portions of 8 behind 1016, {sizes}"] = (
            lambda qd=qd, od=od, kc=kc, vc=vc, table=table, rel=rel, talk=talk, gate=gate, pk=pk: M.talk_paged(
                qd, kc, vc, table, od, talk, short, keys=1024, gate=gate, bias=rel, splits=2, **pk), 4.0 * B * H * D * 1024, 32 * 1024 * G * D * 4)
        cases[f"like: paged_window_prefill, 32 portions of 8 behind 1016, {sizes}"] = (
            lambda qd=qd, od=od, kc=kc, vc=vc, table=table, pk=pk: M.paged_window_attention(qd, kc, vc, table, od, short, **pk),
            4.0 * B * H * D * 1024, 32 * 1024 * G * D * 4)
    up, bias, act = rn(4 * W, W, s=0.02), rn(4 * W), None
    for n in (N, 64):
        few = dict(split_k=0, block_n=128) if n < 256 else {}
        for act, like in (("relu2", ""), ("gelu", "like: ")):
            cases[f"{like}gemm + bias + {act} {n} x 8192 x 2048"] = (
                lambda n=n, act=act, few=few: K.gemm(h[:n], up, bias=bias, act=act, deterministic=True, **few), 2.0 * n * W * 4 * W, 8 * W * W)
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
