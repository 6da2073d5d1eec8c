"""Serving decoders with heterogeneous layers (`lm.hybrid`) on the shared engine.

What differs from the GPT-2 family is below `Engine.forward`: the layer loop, and what a sequence owns beside its cache
pages.  Pages exist for the layers with attention only (keys and values may have different widths); the layers with a
recurrence or a short convolution keep one slot per sequence: the FP32 state and the last inputs of the convolution.  A sequence that
starts over starts from zeros because its first segment starts at position 0, so a slot needs no clearing when it is used
again.

A step runs every row of the batch through each projection together; the mixers then take the segments of the batch (one
per sequence) in up to three groups, one-token segments, short ones and long ones, with the kernel that suits each:

* attention: split-key decode kernel | paged prompt kernel | tcgen05 flash kernel (fresh prompts, head sizes 64 / 128)
* recurrences: token-by-token kernel with the state tile in shared memory | chunked tensor-core kernel
* latent attention: `latent`; attention over convolved projections: `conv_attention`; attention on normed queries and keys:
  `normed_attention`; gated linear attention: `gla`; feed-forwards of experts: `experts`; the long segments of a step on the prompt kernels: `prompt`

The residual stream is FP32; one kernel adds a sublayer output (normed or not) to it and prepares it for the next sublayer, also where
the residual is several streams.  A layer that runs several times has a cache of its own for every run.  In FP32 precision the same layer loop runs the kernels' FP32 forms and plain FP32 matrix products.
"""
from __future__ import annotations

from dataclasses import astuple
from typing import Dict, List, Optional, Sequence

import torch

from ..lm.config import RopeScaling
from ..lm.hybrid import (GLU_ACTS, PLAIN_ACTS, ConvAttentionSpec, DeltaSpec, GlaSpec, HybridConfig, HybridWeights, LatentSpec,
                         NormedAttentionSpec, ParallelSpec)
from ..lm.rope import rope_inv_freq
from . import conv_attention, experts, gla, latent, normed_attention, prompt
from .engine import Chunk, Engine, _Linear

__all__ = ["HybridEngine"]

FLASH_MIN = 128          # fresh prompts from this length on take the tcgen05 flash kernel where the head size allows it


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class HybridEngine(Engine):
    SEGMENT_ROWS = 4

    # ----------------------------------------------------------------------------- configuration
    def _configure(self, weights: HybridWeights) -> None:
        cfg = self.cfg
        if self.dev.type != "cuda":
            raise ValueError("this model runs on the CUDA kernels only (device 'cuda')")
        if self.tp > 1:
            raise ValueError("this model has no tensor-parallel form")
        if cfg.quant.weights != "bf16" or cfg.quant.kv != "bf16":
            raise ValueError("this model has no quantised weights or cache")
        from ..ops import _cuda as K
        K.lib()
        if not self.fast:
            torch.backends.cuda.matmul.allow_tf32 = False
        self.model: HybridConfig = weights.config
        self.runs = self.model.runs               # the layers in the order they run, some of them several times
        self.L, self.d, self.V = len(self.runs), self.model.width, self.model.vocab
        for i, layer in enumerate(self.model.layers):
            m = layer.mixer
            if self.fast and isinstance(m, ParallelSpec) and max(m.left.dim, m.left.vdim) > 256:
                raise ValueError(f"layer {i}: the BF16 attention kernels take head sizes up to 256")
            if isinstance(m, LatentSpec):
                latent.check(self, i, m)
            if isinstance(m, ConvAttentionSpec):
                conv_attention.check(self, i, m)
            if isinstance(m, NormedAttentionSpec):
                normed_attention.check(self, i, m)
            if layer.experts and layer.experts.shared and self.model.pre_norm:
                raise ValueError(f"layer {i}: the gate of the shared expert reads the residual stream, which this design norms first")
        self.adt = torch.bfloat16 if self.fast else torch.float32
        self.kv_kind = 0
        elem = 2 if self.fast else 4
        self._kv_tok_bytes = max(1, self.model.kv_bytes_per_token(elem))
        self.n_blocks = self._pool_blocks(self._kv_tok_bytes)
        self.ctx = cfg.context if cfg.context > 0 else self.n_blocks * cfg.block_size
        if self.model.positions:
            self.ctx = min(self.ctx, self.model.positions)
        self._rope: Dict[tuple, tuple] = {}
        self._short_len = 16 if self.fast else 1 << 30
        mixers = [layer.mixer for layer in self.model.layers]
        self._prompt_windows = {prompt.Window(m.window) for m in mixers if isinstance(m, LatentSpec) and latent.expandable(m)} | {
            conv_attention.window(m) for m in mixers if isinstance(m, ConvAttentionSpec) and conv_attention.promptable(m)} | {
            normed_attention.window(m) for m in mixers if isinstance(m, NormedAttentionSpec) and normed_attention.promptable(m)}
        self._prompt_slices = normed_attention.slices(mixers)

    def _rope_tables(self, dims: int, base: float, scaling: Optional[RopeScaling] = None):
        """cos / sin [ctx, dims / 2]: angles in double, kept in FP32."""
        scaling = scaling or RopeScaling()
        key = (dims, base, astuple(scaling))
        if key not in self._rope:
            freq, mul = rope_inv_freq(max(dims, 1), base, scaling, self.ctx, dtype=torch.float64)
            ang = torch.arange(self.ctx, dtype=torch.float64)[:, None] * freq[None, : dims // 2]
            self._rope[key] = tuple((f(ang) * mul).float().to(self.dev).contiguous() for f in (torch.cos, torch.sin))
        return self._rope[key]

    # ----------------------------------------------------------------------------- weights
    def _pack(self, parts: Sequence[torch.Tensor], bias: Optional[torch.Tensor] = None):
        """Stacks projections of one input: rows of each part padded to a multiple of 8, columns padded to a multiple of
        8 (``bias``: that of a single part).  Returns the linear layer and the first output column of every part."""
        k = _pad8(parts[0].shape[1])
        offsets, n = [], 0
        for p in parts:
            offsets.append(n)
            n += _pad8(p.shape[0])
        w = torch.zeros((n, k))
        for p, o in zip(parts, offsets):
            w[o: o + p.shape[0], : p.shape[1]] = p.float()
        if bias is not None:
            bias = torch.nn.functional.pad(bias.float(), (0, n - bias.shape[0]))
        lin = _Linear(w, bias, self.dev, self.fast)
        self.weight_nbytes += lin.nbytes
        return lin, offsets

    def _f32(self, t: torch.Tensor) -> torch.Tensor:
        return t.to(self.dev, torch.float32).contiguous()

    def _load(self, weights: HybridWeights) -> None:
        t, model = weights.tensors, self.model
        self.weight_nbytes = 0
        head = torch.zeros((self.Vp, self.d))
        head[: self.V] = t["head"].float()
        self.head, _ = self._pack([head])
        self.embed = t["embed"].to(self.dev, self.adt).contiguous()
        self.side_embed = t["side.embed"].to(self.dev, self.adt).contiguous() if model.token_side else None
        self.pos_embed = t["pos"].to(self.dev, self.adt).contiguous() if model.positions else None
        self.weight_nbytes += sum(e.numel() * e.element_size() for e in (self.embed, self.side_embed, self.pos_embed) if e is not None)
        self.final_norm = self._f32(t["final.norm"]) + model.norm_offset
        self.layers: List[dict] = []
        for i, layer in enumerate(model.layers):
            p, m = f"l{i}.", layer.mixer
            # the norms of the two sublayers: on the input (where the design has it) and on the output
            out = {}
            for k, needed in (("1", True), ("2", bool(layer.ff or layer.experts))):
                if needed:
                    out["pre" + k] = self._f32(t[p + "norm" + k]) + model.norm_offset if model.pre_norm else None
                    name = p + "norm" + k + ("b" if model.pre_norm else "")
                    out["post" + k] = self._f32(t[name]) + model.norm_offset if model.post_norm else None
                    if model.streams:
                        out["hc" + k] = {n: self._f32(t[p + f"hc{k}.{n}"]) for n in ("in", "out", "mix")}
            module = {LatentSpec: latent, ConvAttentionSpec: conv_attention, NormedAttentionSpec: normed_attention,
                      GlaSpec: gla}.get(type(m))
            if module is not None:
                out["mix"] = module.load(self, m, lambda n: t[p + "mix." + n])
            elif isinstance(m, ParallelSpec):
                a, r = m.left, m.right
                w_in = t[p + "mix.right.in"]
                z, xbc, dt = w_in.split([r.inner, r.channels, r.heads], 0)
                left = [t[p + f"mix.left.{n}"] for n in ("q", "k", "v")]
                out["in"], out["off"] = self._pack([*left, z, xbc, dt])
                # both output projections read one buffer [attention | ssd]
                na, nr = a.heads * a.vdim, r.inner
                wo = torch.zeros((_pad8(self.d), _pad8(na) + _pad8(nr)))
                wo[: self.d, :na] = t[p + "mix.left.o"].float()
                wo[: self.d, _pad8(na): _pad8(na) + nr] = t[p + "mix.right.o"].float()
                out["out"] = _Linear(wo, None, self.dev, self.fast)
                self.weight_nbytes += out["out"].nbytes
                out["conv"] = self._f32(t[p + "mix.right.conv"].t())
                out["conv_b"] = self._f32(t[p + "mix.right.conv.b"])
                for n, key in (("dt_bias", "dt_bias"), ("A_log", "a_log"), ("D", "d_skip"), ("norm", "norm")):
                    out[key] = self._f32(t[p + "mix.right." + n])
                out["rope"] = self._rope_tables(a.rope_dims, a.rope_base)
            else:
                # q, k and v stay adjacent (they share one convolution); then b, a and the output gate
                qkv = torch.cat([t[p + f"mix.{n}"] for n in ("q", "k", "v")], 0)
                out["in"], out["off"] = self._pack([qkv, t[p + "mix.b"], t[p + "mix.a"], t[p + "mix.g"]])
                out["out"], _ = self._pack([t[p + "mix.o"]])
                out["conv"] = self._f32(torch.cat([t[p + f"mix.{n}.conv"] for n in ("q", "k", "v")], 0).t())
                out["conv_b"] = None
                for n, key in (("dt_bias", "dt_bias"), ("A_log", "a_log"), ("norm", "norm")):
                    out[key] = self._f32(t[p + "mix." + n])
            if layer.experts:
                out["ff"] = experts.load(self, layer.experts, lambda n: t[p + "mlp." + n])
            if layer.ff and layer.act in PLAIN_ACTS:
                for n in ("up", "down"):
                    out[n], _ = self._pack([t[p + "mlp." + n]], bias=t[p + f"mlp.{n}.b"] if layer.ff_bias else None)
            elif layer.ff:
                out["up"], _ = self._pack([experts.in_turns(t[p + "mlp.gate"], t[p + "mlp.up"])])
                out["down"], _ = self._pack([t[p + "mlp.down"]])
            if model.token_side:
                out["side_gate"], _ = self._pack([t[p + "side.gate"]])
                out["side_proj"], _ = self._pack([t[p + "side.proj"]])
                out["side_norm"] = self._f32(t[p + "side.norm"])
            self.layers.append(out)
        self.layers = [self.layers[i] for i in model.order]

    # ----------------------------------------------------------------------------- cache pages and state slots
    def _alloc_kv(self) -> None:
        cfg = self.cfg
        self.max_blocks = -(-self.ctx // cfg.block_size)
        self.k_cache: list = [None] * self.L
        self.v_cache: list = [None] * self.L
        self.state: list = [None] * self.L        # FP32 [slots, heads, key size, value size]
        self.conv_tail: list = [None] * self.L    # [slots, taps - 1, channels]
        for i, layer in enumerate(self.runs):
            m = layer.mixer
            if isinstance(m, ConvAttentionSpec):
                conv_attention.alloc(self, i, m)
                continue
            if isinstance(m, NormedAttentionSpec):
                normed_attention.alloc(self, i, m)
                continue
            if isinstance(m, GlaSpec):
                self.state[i] = torch.zeros((cfg.max_seqs, m.heads, m.dim, m.vdim), dtype=torch.float32, device=self.dev)
                continue
            if isinstance(m, LatentSpec):     # one row per token, whose leading columns are the values; the padding stays zero
                row = latent.LatentShape(m).row
                self.k_cache[i] = torch.zeros((self.n_blocks, cfg.block_size, 1, row), dtype=self.adt, device=self.dev)
                continue
            if isinstance(m, ParallelSpec):
                a, r = m.left, m.right
                self.k_cache[i] = torch.zeros((self.n_blocks, cfg.block_size, a.kv_heads, a.dim), dtype=self.adt, device=self.dev)
                self.v_cache[i] = torch.zeros((self.n_blocks, cfg.block_size, a.kv_heads, a.vdim), dtype=self.adt, device=self.dev)
                shape, taps, channels = (r.heads, r.state, r.vdim), r.conv, r.channels
            else:
                shape, taps, channels = (m.heads, m.dim, m.vdim), m.conv, m.channels
            self.state[i] = torch.zeros((cfg.max_seqs, *shape), dtype=torch.float32, device=self.dev)
            self.conv_tail[i] = torch.zeros((cfg.max_seqs, max(taps - 1, 1), channels), dtype=self.adt, device=self.dev)
        self.k_scale = self.v_scale = [None] * self.L

    def state_bytes_per_sequence(self) -> int:
        return sum(t[0].numel() * t.element_size() for t in (*self.state, *self.conv_tail) if t is not None)

    def _fork_state(self, src: int, dst: int) -> None:
        for t in (*self.state, *self.conv_tail):
            if t is not None:
                t[dst].copy_(t[src])

    def _check_truncate(self, seq: int, length: int) -> None:
        if self.model.recurrent and 0 < length < self.length(seq):
            raise ValueError("a recurrent state cannot be taken back: truncate to 0, or fork the sequence beforehand")

    def _check_batch(self, chunks: Sequence[Chunk]) -> None:
        seen, last = set(), None
        for c in chunks:
            if c.seq != last and c.seq in seen:
                raise ValueError("chunks of one sequence must be adjacent in a step")
            seen.add(c.seq)
            last = c.seq

    def forward(self, chunks: Sequence[Chunk], layers: int = -1, device_tokens: bool = False) -> torch.Tensor:
        if self.model.recurrent and 0 <= layers < self.L:
            raise ValueError("running the first layers only would advance some states and not others")
        return super().forward(chunks, layers, device_tokens)

    # ----------------------------------------------------------------------------- one step
    def _body_rows(self, dv: torch.Tensor, logit_rows: int, runs, nl: int) -> torch.Tensor:
        from ..ops import _mixers as M
        table = dv[self.INDEX_ROWS:]
        groups, first = [], 0
        for count, longest, total in self._segments:
            groups.append(M.Segments(table, first, count, longest, total))
            first += count
        self._groups = groups
        single, short, long_ = groups
        self._many = M.Segments(table, single.count, short.count + long_.count, max(short.max_len, long_.max_len),
                                short.total + long_.total)
        self._stepped = M.Segments(table, 0, single.count + short.count, max(single.max_len, short.max_len),
                                   single.total + short.total)
        self._every = M.Segments(table, 0, first, max(g.max_len for g in groups), sum(g.total for g in groups))
        prompt.plan(self, self._prompt_windows, self._prompt_slices)
        return self._body(dv[0], dv[1], dv[2], dv[3], dv[4], dv[5][:logit_rows], runs, nl)

    def _buffer(self, rows: int, cols: int) -> torch.Tensor:
        """Activation buffer whose pitch the tensor-core GEMM accepts; columns past ``cols`` are zeros."""
        ld = _pad8(cols)
        return (torch.zeros if ld != cols else torch.empty)((rows, ld), dtype=self.adt, device=self.dev)

    def _most_keys(self, a) -> int:
        """The most keys a row can see."""
        sizes = [n for n in (a.window, getattr(a, "chunk", 0)) if n > 0]
        return min(min(sizes) + getattr(a, "keep_first", 0), self.ctx) if sizes else self.ctx

    def _decode_splits(self, a, rows: int) -> int:
        if self.cfg.decode_splits > 0:
            return self.cfg.decode_splits
        keys = self._most_keys(a)
        ctas = rows * a.kv_heads * (-(-(a.heads // a.kv_heads) // 16))
        return max(1, min(592 // max(ctas, 1), -(-keys // 256), 32))

    def _attention(self, i: int, a, proj, off, out, out_scale: float) -> None:
        """Rotated queries in ``proj`` against the cache of layer ``i``; ``out``: [rows, heads * vdim] view."""
        from ..ops import _cuda as K
        from ..ops import _mixers as M
        single, short, long_ = self._groups
        q = proj[:, off: off + a.heads * a.dim]
        kw = dict(heads=a.heads, block_size=self.cfg.block_size, window=a.window, scale=a.scale, softcap=a.softcap,
                  out_scale=out_scale)
        paged = (self.k_cache[i], self.v_cache[i], self.block_table, out)
        if not self.fast:
            M.paged_window_attention(q, *paged, self._every, **kw)
            return
        if single.count:
            M.paged_window_attention(q, *paged, single, splits=self._decode_splits(a, single.count), **kw)
        if not self._many.count:
            return
        host = self._host_rows[self.INDEX_ROWS:]
        flash = long_.count > 0 and a.dim == a.vdim and a.dim in (64, 128) and a.scale > 0 and self._many.count <= 64 and all(
            int(host[1, j]) >= FLASH_MIN and int(host[2, j]) == 0 for j in range(single.count, single.count + self._many.count))
        if not flash:
            M.paged_window_attention(q, *paged, self._many, **kw)
            return
        _, k0, v0 = self.layers[i]["off"][:3]
        for j in range(single.count, single.count + self._many.count):
            r0, n = int(host[0, j]), int(host[1, j])
            rows = proj[r0: r0 + n]
            K.attention_fwd(rows[:, off: off + a.heads * a.dim].view(1, n, a.heads, a.dim),
                            rows[:, k0: k0 + a.kv_heads * a.dim].view(1, n, a.kv_heads, a.dim),
                            rows[:, v0: v0 + a.kv_heads * a.vdim].view(1, n, a.kv_heads, a.vdim), causal=True,
                            window=a.window, scale=a.scale, softcap=a.softcap, out_scale=out_scale,
                            out=out[r0: r0 + n].view(1, n, a.heads, a.vdim))

    def _conv(self, x, w, bias, tail) -> torch.Tensor:
        from ..ops import _mixers as M
        y = torch.empty((x.shape[0], _pad8(w.shape[1])), dtype=self.adt, device=self.dev)[:, : w.shape[1]]
        for seg in (self._groups[0], self._many):
            if seg.count:
                M.conv_silu(x, y, w, bias, tail, seg)
        return y

    def _parallel_mixer(self, i: int, m: ParallelSpec, lw: dict, h, pos, slot) -> torch.Tensor:
        from ..ops import _mixers as M
        a, r, n = m.left, m.right, h.shape[0]
        proj = self._linear(h, lw["in"])
        oq, ok, ov, oz, ox, od = lw["off"]
        M.rope_append(proj, oq, ok, ov, a.heads, a.kv_heads, a.dim, a.vdim, a.rope_dims, pos, slot, *lw["rope"],
                      self.k_cache[i], self.v_cache[i])
        na, nr = a.heads * a.vdim, r.inner
        ka = _pad8(na)
        both = (torch.empty if ka == na and nr % 8 == 0 else torch.zeros)((n, ka + _pad8(nr)), dtype=self.adt, device=self.dev)
        self._attention(i, a, proj, oq, both[:, :na], m.left_scale)
        xbc = self._conv(proj[:, ox: ox + r.channels], lw["conv"], lw["conv_b"], self.conv_tail[i])
        y = torch.empty((n, nr), dtype=self.adt, device=self.dev)
        ssd = (xbc, proj[:, od: od + r.heads], y, lw["dt_bias"], lw["a_log"], lw["d_skip"], self.state[i], r.groups)
        stepped, chunked = self._recurrence_groups(r.state)
        if stepped.count:
            M.ssd(*ssd, stepped)
        if chunked is not None:
            M.ssd(*ssd, chunked, chunked=True, parts=self._ssd_parts(r))
        M.gated_norm(y, proj[:, oz: oz + nr], lw["norm"], both[:, ka: ka + nr], groups=r.norm_groups, gate_first=True,
                     eps=self.model.norm_eps, out_scale=m.right_scale)
        return self._linear(both, lw["out"])

    def _recurrence_groups(self, key_size: int):
        """The segments that run token by token, and those that run in chunks (None: no such segments)."""
        from ..ops import _mixers as M
        if self._groups[2].count == 0 or key_size > M.CHUNK_MAX_KEY:
            return self._every, None
        return self._stepped, self._groups[2]

    def _ssd_parts(self, r) -> int:
        """Spans per long segment: enough (segment, head, span) blocks to fill the GPU, at least 4 chunks each."""
        seg = self._groups[2]
        chunks = -(-seg.max_len // 64)
        return max(1, min(296 // max(1, seg.count * r.heads), chunks // 4))

    def _delta_mixer(self, i: int, m: DeltaSpec, lw: dict, h) -> torch.Tensor:
        from ..ops import _mixers as M
        n = h.shape[0]
        proj = self._linear(h, lw["in"])
        ox, ob, oa, og = lw["off"]
        qkv = self._conv(proj[:, ox: ox + m.channels], lw["conv"], lw["conv_b"], self.conv_tail[i])
        o = torch.empty((n, m.heads * m.vdim), dtype=self.adt, device=self.dev)
        args = (qkv, proj[:, ob: ob + m.heads], proj[:, oa: oa + m.heads], o, lw["dt_bias"], lw["a_log"], self.state[i], m.kv_heads)
        kw = dict(unit_eps=m.unit_eps, q_scale=m.dim ** -0.5)
        stepped, chunked = self._recurrence_groups(m.dim)
        if stepped.count:
            M.delta(*args, stepped, **kw)
        if chunked is not None:
            M.delta(*args, chunked, chunked=True, **kw)
        out = self._buffer(n, m.heads * m.vdim)
        M.gated_norm(o, proj[:, og: og + m.heads * m.vdim], lw["norm"], out[:, : m.heads * m.vdim], groups=m.heads,
                     gate_first=False, eps=self.model.norm_eps)
        return self._linear(out, lw["out"])

    def _gated(self, h, lin: _Linear, glu) -> torch.Tensor:
        """Gated activation of a product whose columns are turns of eight gates and eight values."""
        from ..ops import _cuda as K
        from ..ops import _mixers as M
        if self.fast and K.gated_gemm_ok(h.shape[0], lin.n):
            return K.gated_gemm(h, lin.w, glu)
        both = self._linear(h, lin)
        act = torch.empty((h.shape[0], lin.n // 2), dtype=self.adt, device=self.dev)
        M.glu(both, act, glu, interleaved=True)
        return act

    def _plain(self, h, lw: dict, act: str) -> torch.Tensor:
        """A feed-forward without a gate."""
        if self.fast:
            return self._linear(self._linear(h, lw["up"], act=act), lw["down"])
        return self._linear(torch.relu(self._linear(h, lw["up"])).square_(), lw["down"])

    def _mixer(self, i: int, m, lw: dict, h, pos, slot) -> torch.Tensor:
        if isinstance(m, LatentSpec):
            return latent.mixer(self, i, m, lw["mix"], h, pos, slot)
        if isinstance(m, ConvAttentionSpec):
            return conv_attention.mixer(self, i, m, lw["mix"], h, slot)
        if isinstance(m, NormedAttentionSpec):
            return normed_attention.mixer(self, i, m, lw["mix"], h, pos, slot)
        if isinstance(m, GlaSpec):
            return gla.mixer(self, i, m, lw["mix"], h)
        if isinstance(m, ParallelSpec):
            return self._parallel_mixer(i, m, lw, h, pos, slot)
        return self._delta_mixer(i, m, lw, h)

    def _body(self, tok, pos, slot, rseq, ctx_len, logit_rows, runs, nl: int) -> torch.Tensor:
        from ..ops import _mixers as M
        n, eps, model, cap = tok.shape[0], self.model.norm_eps, self.model, self._capture
        mult = model.residual_mult
        streams = model.streams
        x = torch.empty((n, streams, self.d) if streams else (n, self.d), dtype=torch.float32, device=self.dev)
        h = torch.empty((n, _pad8(self.d)), dtype=self.adt, device=self.dev)
        routes = experts.route(self, tok)

        # one kernel between two sublayers: `took(lw, k)` says how the output of sublayer k of a layer joins the residual, `feed(lw, k)`
        # what sublayer k reads of it
        residual = M.stream_residual if streams else M.residual_norm

        def feed(lw, k: str) -> dict:
            norm = lw["pre" + k]
            if streams:
                return {"w_next": norm, "h": h, "read": lw["hc" + k]["in"]}
            return {"w_next": norm, "h": h} if norm is not None else {"x_cast": h}

        def took(lw, k: str) -> dict:
            if streams:
                return {"mix": lw["hc" + k]["mix"], "out": lw["hc" + k]["out"]}
            return {"w_post": lw["post" + k], "res_mult": mult}
        residual(x, tokens=tok, table=self.embed, eps=eps, embed_scale=model.embed_scale, positions=pos, pos_table=self.pos_embed,
                 **feed(self.layers[0], "1"))
        for i, (layer, lw) in enumerate(zip(self.runs[:nl], self.layers)):
            more = feed(self.layers[i + 1], "1") if i + 1 < nl else {}
            after = more if not model.token_side else {"x_cast": h}
            y, add = self._mixer(i, layer.mixer, lw, h, pos, slot), took(lw, "1")
            if layer.experts:
                f, ff, r = layer.experts, lw["ff"], routes[i]
                extra, by_slot = {}, None
                if f.shared:
                    gate = torch.empty(n, dtype=torch.float32, device=self.dev)
                    extra.update(w_dot=ff["sg"], dot_out=gate)
                if r is not None and r.align >= 128:
                    by_slot = torch.empty((r.max_slots, h.shape[1]), dtype=self.adt, device=self.dev)
                    extra.update(scatter=by_slot, slots=r.slots, top=r.top)
                residual(x, y=y, eps=eps, **add, **feed(lw, "2"), **extra)
                if f.router:
                    r, by_slot = experts.gate(self, f, ff, h)
                rows, y = experts.forward(self, f, ff, r, h, by_slot)
                add = {**took(lw, "2"), "experts": rows, "slots": r.slots, "top": r.top,
                       "weights": r.weight, "y_gate": gate if f.shared else None}
            elif layer.ff:
                residual(x, y=y, eps=eps, **add, **feed(lw, "2"))
                if layer.act in PLAIN_ACTS:
                    y = self._plain(h, lw, layer.act)
                else:
                    y = self._linear(self._gated(h, lw["up"], M.Glu(GLU_ACTS.index(layer.act))), lw["down"])
                add = took(lw, "2")
            residual(x, y=y, eps=eps, **add, **after)
            if model.token_side:
                gate = self._linear(h, lw["side_gate"], out_dtype=torch.float32)
                side = torch.empty(gate.shape, dtype=self.adt, device=self.dev)
                M.token_side_gate(gate, tok, self.side_embed, i * model.token_side, side, model.token_side)
                y = self._linear(side, lw["side_proj"])
                M.residual_norm(x, y=y, w_post=lw["side_norm"], eps=eps, res_mult=mult, **more)
            if cap is not None:
                cap.append((x.sum(1) if streams else x.detach()).float().cpu())
        if logit_rows.shape[0] == 0:
            return torch.zeros((0, self.Vp), dtype=torch.float32, device=self.dev)
        xr = x.index_select(0, logit_rows.long())
        hr = torch.empty((xr.shape[0], _pad8(self.d)), dtype=self.adt, device=self.dev)
        residual(xr, w_next=self.final_norm, h=hr, eps=eps)
        logits = self._linear(hr, self.head, out_dtype=torch.float32)
        if model.logit_softcap > 0 or model.logit_scale != 1.0:
            M.softcap_(logits, self.V, model.logit_softcap, model.logit_scale)
        return logits
