"""ctypes bindings of the mixer kernels (``nx_api_mixers.h``): the residual / norm chain, rotary embedding with cache
append, windowed soft-capped paged attention, the short causal convolution, the SSD, gated-delta and gated-linear
recurrences, gated norms, gated activations and the per-layer token input.  BF16 or FP32 activations; every wrapper launches on the current torch stream."""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass
from typing import Optional

import torch

from . import _cuda as K
from ._cuda import Glu

CHUNK = 64            # tokens per chunk of the tensor-core recurrences
CHUNK_MAX_KEY = 256   # their largest state size along the key dimension


class SegmentArgs(C.Structure):
    _fields_ = [("row0", C.c_void_p), ("len", C.c_void_p), ("pos", C.c_void_p), ("seq", C.c_void_p),
                ("count", C.c_int32), ("max_len", C.c_int32), ("total_len", C.c_int32)]


class ResidualNormArgs(C.Structure):
    _fields_ = [("x", C.c_void_p), ("tokens", C.c_void_p), ("table", C.c_void_p), ("y", C.c_void_p), ("w_post", C.c_void_p),
                ("w_next", C.c_void_p), ("h", C.c_void_p), ("x_cast", C.c_void_p), ("ldy", C.c_int64), ("ldh", C.c_int64),
                ("rows", C.c_int32), ("cols", C.c_int32), ("dtype", C.c_int32), ("eps", C.c_float), ("embed_scale", C.c_float),
                ("res_mult", C.c_float), ("experts", C.c_void_p), ("expert_slots", C.c_void_p), ("y_gate", C.c_void_p),
                ("ld_experts", C.c_int64), ("top", C.c_int32), ("expert_scale", C.c_float), ("w_dot", C.c_void_p),
                ("dot_out", C.c_void_p), ("scatter", C.c_void_p), ("scatter_slots", C.c_void_p), ("expert_weights", C.c_void_p),
                ("positions", C.c_void_p), ("pos_table", C.c_void_p)]


class StreamResidualArgs(C.Structure):
    _fields_ = [("x", C.c_void_p), ("tokens", C.c_void_p), ("table", C.c_void_p), ("positions", C.c_void_p), ("pos_table", C.c_void_p),
                ("y", C.c_void_p), ("mix", C.c_void_p), ("out", C.c_void_p), ("in_", C.c_void_p), ("w_next", C.c_void_p),
                ("h", C.c_void_p), ("ldy", C.c_int64), ("ldh", C.c_int64), ("rows", C.c_int32), ("cols", C.c_int32),
                ("streams", C.c_int32), ("dtype", C.c_int32), ("eps", C.c_float), ("embed_scale", C.c_float)]


class HeadPrepArgs(C.Structure):
    _fields_ = [("proj", C.c_void_p), ("ld", C.c_int64), ("q_off", C.c_int32), ("k_off", C.c_int32), ("v_off", C.c_int32),
                ("g_off", C.c_int32), ("rows", C.c_int32), ("heads", C.c_int32), ("kv_heads", C.c_int32), ("dim", C.c_int32),
                ("vdim", C.c_int32), ("norm_dim", C.c_int32), ("norm_vdim", C.c_int32), ("norm_all", C.c_int32),
                ("unit_values", C.c_int32), ("store_kv", C.c_int32), ("every", C.c_int32), ("dtype", C.c_int32), ("eps", C.c_float),
                ("q_scale", C.c_float), ("coef", C.c_float), ("w_q", C.c_void_p), ("w_k", C.c_void_p), ("head_scale", C.c_void_p),
                ("positions", C.c_void_p), ("slots", C.c_void_p), ("k_cache", C.c_void_p), ("v_cache", C.c_void_p),
                ("gate", C.c_void_p)]


class LatentPrepArgs(C.Structure):
    _fields_ = [("proj", C.c_void_p), ("ld", C.c_int64), ("q_off", C.c_int32), ("c_off", C.c_int32), ("r_off", C.c_int32),
                ("g_off", C.c_int32), ("rows", C.c_int32), ("q_rank", C.c_int32), ("kv_rank", C.c_int32), ("rot_dims", C.c_int32),
                ("heads", C.c_int32), ("dtype", C.c_int32), ("eps", C.c_float), ("w_q", C.c_void_p), ("w_kv", C.c_void_p),
                ("positions", C.c_void_p), ("slots", C.c_void_p), ("cos_t", C.c_void_p), ("sin_t", C.c_void_p), ("cq", C.c_void_p),
                ("ldq", C.c_int64), ("cache", C.c_void_p), ("ld_cache", C.c_int64), ("rot_col", C.c_int32), ("lat", C.c_void_p),
                ("gate", C.c_void_p)]


class RopeAppendArgs(C.Structure):
    _fields_ = [("proj", C.c_void_p), ("ld", C.c_int64), ("q_off", C.c_int32), ("k_off", C.c_int32), ("v_off", C.c_int32),
                ("rows", C.c_int32), ("heads", C.c_int32), ("kv_heads", C.c_int32), ("dim", C.c_int32), ("vdim", C.c_int32),
                ("rot_dims", C.c_int32), ("dtype", C.c_int32), ("positions", C.c_void_p), ("slots", C.c_void_p),
                ("cos_t", C.c_void_p), ("sin_t", C.c_void_p), ("k_cache", C.c_void_p), ("v_cache", C.c_void_p)]


class ConvArgs(C.Structure):
    _fields_ = [("x", C.c_void_p), ("y", C.c_void_p), ("w", C.c_void_p), ("bias", C.c_void_p), ("state", C.c_void_p),
                ("ldx", C.c_int64), ("ldy", C.c_int64), ("channels", C.c_int32), ("taps", C.c_int32), ("dtype", C.c_int32),
                ("seg", SegmentArgs)]


class ConvRopeArgs(C.Structure):
    _fields_ = [("conv", ConvArgs), ("heads", C.c_int32), ("kv_heads", C.c_int32), ("dim", C.c_int32), ("vdim", C.c_int32),
                ("rot_dims", C.c_int32), ("store_kv", C.c_int32), ("slots", C.c_void_p), ("cos_t", C.c_void_p), ("sin_t", C.c_void_p),
                ("k_cache", C.c_void_p), ("v_cache", C.c_void_p), ("mix", C.c_void_p), ("first", C.c_void_p)]


class GlaArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("decay", C.c_void_p), ("o", C.c_void_p),
                ("state", C.c_void_p), ("ld", C.c_int64), ("ld_decay", C.c_int64), ("ldo", C.c_int64), ("heads", C.c_int32),
                ("dim", C.c_int32), ("vdim", C.c_int32), ("dtype", C.c_int32), ("q_scale", C.c_float), ("seg", SegmentArgs),
                ("part_state", C.c_void_p), ("part_decay", C.c_void_p), ("parts", C.c_int32), ("span", C.c_int32)]


class SsdArgs(C.Structure):
    _fields_ = [("xbc", C.c_void_p), ("dt", C.c_void_p), ("y", C.c_void_p), ("dt_bias", C.c_void_p), ("a_log", C.c_void_p),
                ("d_skip", C.c_void_p), ("state", C.c_void_p), ("ld_xbc", C.c_int64), ("ld_dt", C.c_int64), ("ldy", C.c_int64),
                ("heads", C.c_int32), ("groups", C.c_int32), ("n_state", C.c_int32), ("vdim", C.c_int32), ("dtype", C.c_int32),
                ("seg", SegmentArgs), ("part_state", C.c_void_p), ("part_decay", C.c_void_p), ("parts", C.c_int32),
                ("span", C.c_int32)]


class DeltaArgs(C.Structure):
    _fields_ = [("qkv", C.c_void_p), ("b", C.c_void_p), ("a", C.c_void_p), ("o", C.c_void_p), ("dt_bias", C.c_void_p),
                ("a_log", C.c_void_p), ("state", C.c_void_p), ("ld_qkv", C.c_int64), ("ld_ba", C.c_int64), ("ldo", C.c_int64),
                ("heads", C.c_int32), ("kv_heads", C.c_int32), ("dim", C.c_int32), ("vdim", C.c_int32), ("dtype", C.c_int32),
                ("unit_eps", C.c_float), ("q_scale", C.c_float), ("seg", SegmentArgs), ("scratch", C.c_void_p)]


class GatedNormArgs(C.Structure):
    _fields_ = [("y", C.c_void_p), ("z", C.c_void_p), ("w", C.c_void_p), ("out", C.c_void_p), ("ldy", C.c_int64),
                ("ldz", C.c_int64), ("ldo", C.c_int64), ("rows", C.c_int32), ("groups", C.c_int32), ("group_size", C.c_int32),
                ("gate_first", C.c_int32), ("w_shared", C.c_int32), ("dtype", C.c_int32), ("eps", C.c_float),
                ("out_scale", C.c_float)]


class PagedWindowArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k_cache", C.c_void_p), ("v_cache", C.c_void_p), ("block_table", C.c_void_p),
                ("out", C.c_void_p), ("ldq", C.c_int64), ("ldo", C.c_int64), ("part_o", C.c_void_p), ("part_ml", C.c_void_p),
                ("heads", C.c_int32), ("kv_heads", C.c_int32), ("dim", C.c_int32), ("vdim", C.c_int32),
                ("block_size", C.c_int32), ("max_blocks", C.c_int32), ("window", C.c_int32), ("splits", C.c_int32),
                ("dtype", C.c_int32), ("scale", C.c_float), ("softcap", C.c_float), ("out_scale", C.c_float),
                ("seg", SegmentArgs), ("k_pitch", C.c_int64), ("v_pitch", C.c_int64), ("gate", C.c_void_p), ("sink", C.c_void_p),
                ("keep_first", C.c_int32), ("chunk", C.c_int32), ("bias_len", C.c_int32), ("all_values", C.c_int32),
                ("bias", C.c_void_p)]


class TalkPagedArgs(C.Structure):
    _fields_ = [("base", PagedWindowArgs), ("talk", C.c_void_p), ("scores", C.c_void_p), ("weights", C.c_void_p), ("pitch", C.c_int64),
                ("rows", C.c_int32)]


class TalkPromptArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("out", C.c_void_p), ("bias", C.c_void_p),
                ("blocks", C.c_void_p), ("status", C.c_void_p), ("ldq", C.c_int64), ("ldk", C.c_int64), ("ldv", C.c_int64),
                ("ldo", C.c_int64), ("n_blocks", C.c_int32), ("q_rows", C.c_int32), ("kv_rows", C.c_int32), ("heads", C.c_int32),
                ("kv_heads", C.c_int32), ("dim", C.c_int32), ("vdim", C.c_int32), ("window", C.c_int32), ("chunk", C.c_int32),
                ("bias_len", C.c_int32), ("bias_pitch", C.c_int32), ("scale", C.c_float)]


class LatentPromptArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("kv", C.c_void_p), ("lat", C.c_void_p), ("out", C.c_void_p), ("gate", C.c_void_p),
                ("blocks", C.c_void_p), ("status", C.c_void_p), ("ldq", C.c_int64), ("ldkv", C.c_int64), ("ld_lat", C.c_int64),
                ("ldo", C.c_int64), ("n_blocks", C.c_int32), ("q_rows", C.c_int32), ("kv_rows", C.c_int32), ("q_head", C.c_int32),
                ("rank", C.c_int32), ("heads", C.c_int32), ("dim", C.c_int32), ("rot", C.c_int32), ("vdim", C.c_int32),
                ("window", C.c_int32), ("scale", C.c_float)]


class WindowPromptArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("out", C.c_void_p), ("sink", C.c_void_p),
                ("blocks", C.c_void_p), ("kept", C.c_void_p), ("status", C.c_void_p), ("ldq", C.c_int64), ("ldk", C.c_int64),
                ("ldv", C.c_int64), ("ldo", C.c_int64), ("n_blocks", C.c_int32), ("q_rows", C.c_int32), ("kv_rows", C.c_int32),
                ("heads", C.c_int32), ("kv_heads", C.c_int32), ("dim", C.c_int32), ("vdim", C.c_int32), ("window", C.c_int32),
                ("keep_first", C.c_int32), ("scale", C.c_float), ("gate", C.c_void_p), ("bias", C.c_void_p), ("bias_len", C.c_int32),
                ("chunk", C.c_int32)]


class LatentAttnArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("cache", C.c_void_p), ("block_table", C.c_void_p), ("out", C.c_void_p), ("gate", C.c_void_p),
                ("part_o", C.c_void_p), ("part_ml", C.c_void_p), ("status", C.c_void_p), ("ldq", C.c_int64), ("ldo", C.c_int64),
                ("heads", C.c_int32), ("row", C.c_int32), ("rank", C.c_int32), ("block_size", C.c_int32), ("max_blocks", C.c_int32),
                ("window", C.c_int32), ("splits", C.c_int32), ("n_slots", C.c_int32), ("scale", C.c_float), ("seg", SegmentArgs)]


LATENT_MAX_RANK, LATENT_MAX_ROW = 512, 768
PROMPT_MAX_BIAS = 3072       # distances of a bias table of the tcgen05 prompt kernels
TALK_MAX_HEADS = 96          # heads that mix their weights
TALK_SCRATCH = 1 << 29       # bytes of scores and weights of one launch of such heads
TALK_WIDE = 1 << 29          # bytes of every head's outputs with the values of every KV head that wait for their mixture at a time
BIAS_MARGIN = 256            # entries of an extended bias table on either side of its distances


@dataclass
class Segments:
    """A range of a device segment table ``[4, width]`` (first row, rows, first position, sequence)."""
    table: torch.Tensor
    first: int
    count: int
    max_len: int
    total: int

    def args(self) -> SegmentArgs:
        t, step = self.table, self.table.stride(0) * 4
        p = t.data_ptr() + self.first * 4
        return SegmentArgs(p, p + step, p + 2 * step, p + 3 * step, self.count, self.max_len, self.total)


def _dt(t: torch.Tensor) -> int:
    return K._DT[t.dtype]


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def residual_norm(x, *, y=None, w_post=None, w_next=None, h=None, x_cast=None, tokens=None, table=None, eps, embed_scale=1.0,
                  res_mult=1.0, experts=None, slots=None, top=0, weights=None, y_gate=None, w_dot=None, dot_out=None,
                  scatter=None, positions=None, pos_table=None) -> None:
    """x (FP32) = embed_scale * table[tokens] (+ pos_table[positions]), or x + res_mult * rms(y) * w_post (without w_post: x + res_mult * y);  h = rms(x) *
    w_next;  x_cast = x in the activation dtype.  With ``experts`` the sublayer output is the mean of the rows
    ``experts[slots[r, :]]``, or their sum with ``weights`` [rows, top] (FP32), + y_gate[r] * y[r].  ``dot_out`` = sigmoid(x .
    w_dot); ``scatter[slots[r, :]]`` = the row of x_cast."""
    lead = next((t for t in (h, x_cast, scatter) if t is not None), None)
    act = next(t for t in (lead, y, experts, table) if t is not None)
    if any(t is not None and t.stride(0) != lead.stride(0) for t in (h, x_cast, scatter)):
        raise ValueError("residual_norm: h, x_cast and scatter must share one row pitch")
    a = ResidualNormArgs(_ptr(x), _ptr(tokens), _ptr(table), _ptr(y), _ptr(w_post), _ptr(w_next), _ptr(h), _ptr(x_cast),
                         y.stride(0) if y is not None else 0, lead.stride(0) if lead is not None else x.shape[1], x.shape[0],
                         x.shape[1], _dt(act), eps, embed_scale, res_mult, _ptr(experts), _ptr(slots), _ptr(y_gate),
                         experts.stride(0) if experts is not None else 0, top, 1.0 / top if top and weights is None else 1.0,
                         _ptr(w_dot), _ptr(dot_out), _ptr(scatter), _ptr(slots), _ptr(weights), _ptr(positions), _ptr(pos_table))
    K._check(K.lib().nx_residual_norm(C.byref(a), K._stream()), "nx_residual_norm")


def stream_residual(x, *, eps, y=None, mix=None, out=None, tokens=None, table=None, embed_scale=1.0, positions=None, pos_table=None,
                    w_next=None, h=None, read=None) -> None:
    """x (FP32 [rows, streams, cols]): every stream = embed_scale * table[tokens] + pos_table[positions], or x_t = sum_s mix[s, t] x_s +
    out[t] y;  h = rms(sum_s read[s] x_s) * w_next (``read`` None: ones)."""
    act = next(t for t in (h, y, table) if t is not None)
    a = StreamResidualArgs(_ptr(x), _ptr(tokens), _ptr(table), _ptr(positions), _ptr(pos_table), _ptr(y), _ptr(mix), _ptr(out),
                           _ptr(read), _ptr(w_next), _ptr(h), y.stride(0) if y is not None else 0, h.stride(0) if h is not None else 0,
                           x.shape[0], x.shape[2], x.shape[1], _dt(act), eps, embed_scale)
    K._check(K.lib().nx_stream_residual(C.byref(a), K._stream()), "nx_stream_residual")


def head_prep(proj, offsets, *, heads, kv_heads, dim, vdim, norm_dim, norm_vdim, eps, w_q, w_k, positions, slots, k_cache, v_cache,
              norm_all=False, unit_values=False, store_kv=False, q_scale=1.0, head_scale=None, coef=0.0, every=0, gate=None) -> None:
    """Norms of q and k, the query's factors, cache append and the output gate, in place in ``proj``; ``offsets``: first columns of q,
    k, v and the gate."""
    a = HeadPrepArgs(_ptr(proj), proj.stride(0), *offsets, proj.shape[0], heads, kv_heads, dim, vdim, norm_dim, norm_vdim,
                     int(norm_all), int(unit_values), int(store_kv), every, _dt(proj), eps, q_scale, coef, _ptr(w_q), _ptr(w_k),
                     _ptr(head_scale), _ptr(positions), _ptr(slots), _ptr(k_cache), _ptr(v_cache), _ptr(gate))
    K._check(K.lib().nx_head_prep(C.byref(a), K._stream()), "nx_head_prep")


def head_mix(wide, talk, gate, out, *, heads, kv_heads, vdim) -> None:
    """out [rows, heads * vdim]: out_h = gate_h sum_g talk[h, g] wide[g, KV head of h]; wide [rows, heads * kv_heads * vdim]."""
    K._check(K.lib().nx_head_mix(K._p(wide), C.c_int64(wide.stride(0)), K._p(talk), K._p(gate), K._p(out), C.c_int64(out.stride(0)),
                                 C.c_int(wide.shape[0]), C.c_int(heads), C.c_int(kv_heads), C.c_int(vdim), C.c_int(_dt(wide)),
                                 K._stream()), "nx_head_mix")


def latent_prep(proj, offsets, q_rank, kv_rank, rot_dims, heads, w_q, w_kv, positions, slots, cos_t, sin_t, cq, cache, rot_col,
                gate, *, eps, lat=None) -> None:
    """``offsets``: first columns of the query latent, the key / value latent, the shared key part and the gate in ``proj``;
    cache [blocks, block_size, row], lat [rows, row] or None, gate FP32 [rows, heads] or None; q_rank 0: no query latent."""
    a = LatentPrepArgs(_ptr(proj), proj.stride(0), *offsets, proj.shape[0], q_rank, kv_rank, rot_dims, heads, _dt(proj), eps,
                       _ptr(w_q), _ptr(w_kv), _ptr(positions), _ptr(slots), _ptr(cos_t), _ptr(sin_t), _ptr(cq),
                       cq.stride(0) if cq is not None else 0,
                       _ptr(cache), cache.shape[-1], rot_col, _ptr(lat), _ptr(gate))
    K._check(K.lib().nx_latent_prep(C.byref(a), K._stream()), "nx_latent_prep")


def rope_heads(src, src_head, src_off, dst, dst_head, dst_off, heads, rot_dims, width, positions, cos_t, sin_t) -> None:
    """Rotates ``rot_dims`` columns of every head of ``src`` [rows, .] into ``dst`` (zeros up to ``width``)."""
    K._check(K.lib().nx_rope_heads(K._p(src), C.c_int64(src.stride(0)), C.c_int(src_head), C.c_int(src_off), K._p(dst),
                                   C.c_int64(dst.stride(0)), C.c_int(dst_head), C.c_int(dst_off), C.c_int(src.shape[0]),
                                   C.c_int(heads), C.c_int(rot_dims), C.c_int(width), K._p(positions), K._p(cos_t), K._p(sin_t),
                                   C.c_int(_dt(src)), K._stream()), "nx_rope_heads")


def rope_append(proj, q_off, k_off, v_off, heads, kv_heads, dim, vdim, rot_dims, positions, slots, cos_t, sin_t, k_cache,
                v_cache) -> None:
    a = RopeAppendArgs(_ptr(proj), proj.stride(0), q_off, k_off, v_off, proj.shape[0], heads, kv_heads, dim, vdim, rot_dims,
                       _dt(proj), _ptr(positions), _ptr(slots), _ptr(cos_t), _ptr(sin_t), _ptr(k_cache), _ptr(v_cache))
    K._check(K.lib().nx_rope_append(C.byref(a), K._stream()), "nx_rope_append")


def conv_silu(x, y, w, bias, state, seg: Segments) -> None:
    """x / y: [rows, channels] views; w: FP32 [taps, channels]; state: [slots, taps - 1, channels]."""
    a = ConvArgs(_ptr(x), _ptr(y), _ptr(w), _ptr(bias), _ptr(state), x.stride(0), y.stride(0), w.shape[1], w.shape[0], _dt(x),
                 seg.args())
    K._check(K.lib().nx_conv_silu(C.byref(a), K._stream()), "nx_conv_silu")


def conv_rope_append(x, y, w, bias, state, seg: Segments, *, heads, kv_heads, dim, vdim, rot_dims, cos_t, sin_t, slots, k_cache,
                     v_cache, store_kv=False, mix=None, first=None) -> None:
    """Convolution over the packed q | k | v columns of ``x``, rotation of neighbouring pairs, value mixing (``mix``: FP32 [1] with
    the values ``first`` [rows, kv_heads * vdim]; without it ``first`` is written) and cache append; ``y`` receives q (and k, v)."""
    a = ConvRopeArgs(ConvArgs(_ptr(x), _ptr(y), _ptr(w), _ptr(bias), _ptr(state), x.stride(0), y.stride(0), w.shape[1], w.shape[0],
                              _dt(x), seg.args()), heads, kv_heads, dim, vdim, rot_dims, int(store_kv), _ptr(slots), _ptr(cos_t),
                     _ptr(sin_t), _ptr(k_cache), _ptr(v_cache), _ptr(mix), _ptr(first))
    K._check(K.lib().nx_conv_rope_append(C.byref(a), K._stream()), "nx_conv_rope_append")


def decay_gate(a, w, bias, tau) -> torch.Tensor:
    """log2(sigmoid(a w^T + bias)) / tau in FP32; w FP32 [cols, rank], a [rows, >= rank]."""
    out = torch.empty((a.shape[0], w.shape[0]), dtype=torch.float32, device=a.device)
    K._check(K.lib().nx_decay_gate(K._p(a), C.c_int64(a.stride(0)), K._p(w), K._p(bias), K._p(out), C.c_int64(out.stride(0)),
                                   C.c_int(a.shape[0]), C.c_int(w.shape[0]), C.c_int(w.shape[1]), C.c_float(tau), C.c_int(_dt(a)),
                                   K._stream()), "nx_decay_gate")
    return out


def _spans(a, seg: Segments, parts: int) -> None:
    chunks = -(-seg.max_len // CHUNK)
    per = -(-chunks // max(1, parts))
    a.span, a.parts = per * CHUNK, -(-chunks // per)


def gla(q, k, v, decay, o, state, seg: Segments, *, q_scale, chunked=False, parts=1) -> None:
    """q, k, v: views of one row pitch; decay: FP32 log2 decays [rows, heads * dim]; state: FP32 [slots, heads, dim, vdim]."""
    _, H, D, Dv = state.shape
    if not q.stride(0) == k.stride(0) == v.stride(0):
        raise ValueError("gla: q, k and v must share one row pitch")
    a = GlaArgs(_ptr(q), _ptr(k), _ptr(v), _ptr(decay), _ptr(o), _ptr(state), q.stride(0), decay.stride(0), o.stride(0), H, D, Dv,
                _dt(q), q_scale, seg.args(), None, None, 1, 0)
    if not chunked:
        K._check(K.lib().nx_gla_step(C.byref(a), K._stream()), "nx_gla_step")
        return
    _spans(a, seg, parts)
    if a.parts > 1:
        a.part_state = K.scratch(seg.count * a.parts * H * D * Dv * 4, "gla_state", q.device).data_ptr()
        a.part_decay = K.scratch(seg.count * a.parts * H * D * 4, "gla_decay", q.device).data_ptr()
    K._check(K.lib().nx_gla_chunk(C.byref(a), K._stream()), "nx_gla_chunk")


def ssd(xbc, dt, y, dt_bias, a_log, d_skip, state, groups, seg: Segments, *, chunked=False, parts=1) -> None:
    """state: FP32 [slots, heads, N, P].  ``chunked``: the tensor-core form; its segments are cut into ``parts`` spans
    that run at the same time."""
    _, H, N, P = state.shape
    a = SsdArgs(_ptr(xbc), _ptr(dt), _ptr(y), _ptr(dt_bias), _ptr(a_log), _ptr(d_skip), _ptr(state), xbc.stride(0),
                dt.stride(0), y.stride(0), H, groups, N, P, _dt(xbc), seg.args(), None, None, 1, 0)
    if not chunked:
        K._check(K.lib().nx_ssd_step(C.byref(a), K._stream()), "nx_ssd_step")
        return
    _spans(a, seg, parts)
    if a.parts > 1:
        a.part_state = K.scratch(seg.count * a.parts * H * N * P * 4, "ssd_state", xbc.device).data_ptr()
        a.part_decay = K.scratch(seg.count * a.parts * H * 4, "ssd_decay", xbc.device).data_ptr()
    K._check(K.lib().nx_ssd_chunk(C.byref(a), K._stream()), "nx_ssd_chunk")


def delta(qkv, b, a, o, dt_bias, a_log, state, kv_heads, seg: Segments, *, unit_eps, q_scale, chunked=False) -> None:
    """state: FP32 [slots, heads, D, Dv]."""
    _, H, D, Dv = state.shape
    if b.stride(0) != a.stride(0):
        raise ValueError("delta: the gate projections must share one row pitch")
    args = DeltaArgs(_ptr(qkv), _ptr(b), _ptr(a), _ptr(o), _ptr(dt_bias), _ptr(a_log), _ptr(state), qkv.stride(0), b.stride(0),
                     o.stride(0), H, kv_heads, D, Dv, _dt(qkv), unit_eps, q_scale, seg.args(), None)
    if chunked:
        size = K.lib().nx_delta_scratch_bytes
        size.restype = C.c_int64
        args.scratch = K.scratch(size(C.c_int(H), C.c_int(seg.count), C.c_int(seg.max_len)), "delta", qkv.device).data_ptr()
    fn = K.lib().nx_delta_chunk if chunked else K.lib().nx_delta_step
    K._check(fn(C.byref(args), K._stream()), "nx_delta_chunk" if chunked else "nx_delta_step")


def gated_norm(y, z, w, out, *, groups, gate_first, eps, out_scale=1.0) -> None:
    """y, z, out: [rows, groups * size] views; w: FP32, one entry per column or [size] shared by the groups."""
    size = y.shape[1] // groups
    a = GatedNormArgs(_ptr(y), _ptr(z), _ptr(w), _ptr(out), y.stride(0), z.stride(0), out.stride(0), y.shape[0], groups, size,
                      int(gate_first), int(groups > 1 and w.numel() == size), _dt(y), eps, out_scale)
    K._check(K.lib().nx_gated_norm(C.byref(a), K._stream()), "nx_gated_norm")


def token_side_gate(a, tokens, table, offset, out, dim) -> None:
    """a: FP32 [rows, >= dim]; table and out in the activation dtype."""
    if a.dtype != torch.float32:
        raise ValueError("token_side_gate: the gate is FP32")
    K._check(K.lib().nx_token_side_gate(K._p(a), C.c_int64(a.stride(0)), K._p(tokens), K._p(table), C.c_int64(table.stride(0)),
                                        C.c_int(offset), K._p(out), C.c_int64(out.stride(0)), C.c_int(a.shape[0]), C.c_int(dim),
                                        C.c_int(_dt(out)), K._stream()), "nx_token_side_gate")


def silu_mul(h, out) -> None:
    """h: [rows, 2 F] = [gate | up]; out: [rows, F]."""
    K._check(K.lib().nx_silu_mul(K._p(h), C.c_int64(h.stride(0)), K._p(out), C.c_int64(out.stride(0)), C.c_int(h.shape[0]),
                                 C.c_int(h.shape[1] // 2), C.c_int(_dt(h)), K._stream()), "nx_silu_mul")


def glu(h, out, kind: Glu, *, interleaved=False) -> None:
    """h: [rows, 2 F], gates and values in two halves or in turns of eight columns; out: [rows, F]."""
    K._check(K.lib().nx_glu(K._p(h), C.c_int64(h.stride(0)), K._p(out), C.c_int64(out.stride(0)), C.c_int(h.shape[0]),
                            C.c_int(h.shape[1] // 2), C.c_int(int(interleaved)), kind, C.c_int(_dt(h)), K._stream()), "nx_glu")


def softcap_(x, cols, cap, scale=1.0) -> None:
    """x = cap * tanh(scale * x / cap) in place (cap 0: x = scale * x)."""
    for r0 in range(0, x.shape[0], 32768):
        part = x[r0: r0 + 32768]
        K._check(K.lib().nx_softcap(K._p(part), C.c_int64(part.stride(0)), C.c_int(part.shape[0]), C.c_int(cols), C.c_float(cap),
                                    C.c_float(scale), K._stream()), "nx_softcap")


def _paged_args(q, k_cache, v_cache, block_table, out, seg, heads, block_size, window, scale, softcap, out_scale, gate, vdim, keep_first,
                sink, chunk, bias, all_values) -> PagedWindowArgs:
    G, D = k_cache.shape[2], k_cache.shape[3]
    if vdim:
        v_cache = k_cache
        if G != 1:
            raise ValueError("paged_window_attention: a latent cache has one KV head")
    Dv = vdim or v_cache.shape[3]
    return PagedWindowArgs(_ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(block_table), _ptr(out), q.stride(0), out.stride(0),
                           None, None, heads, G, D, Dv, block_size, block_table.shape[1], window, 1, _dt(q), scale, softcap, out_scale,
                           seg.args(), k_cache.stride(1), v_cache.stride(1), _ptr(gate), _ptr(sink), keep_first, chunk,
                           bias.shape[1] if bias is not None else 0, int(all_values), _ptr(bias))


def paged_window_attention(q, k_cache, v_cache, block_table, out, seg: Segments, *, heads, block_size, window, scale,
                           softcap=0.0, out_scale=1.0, splits=1, gate=None, vdim=0, keep_first=0, sink=None, chunk=0, bias=None,
                           all_values=False) -> None:
    """q: [rows, heads * dim] view; caches [blocks, block_size, kv_heads, dim | vdim]; out [rows, heads * vdim] view.
    One-row segments run the decode kernel, longer ones the prompt kernel (BF16); FP32 has one kernel for both.
    ``vdim`` > 0: a latent cache, the values are the leading ``vdim`` columns of the keys (``v_cache`` is not used).
    ``gate``: FP32 [rows, heads] factor of the output.  ``keep_first``: the first keys stay visible; ``sink``: FP32 [heads], a
    score that counts in the denominator only.  ``chunk``: only keys of the row's chunk of positions; ``bias``: FP32 [heads, distances],
    the last one for all beyond; ``all_values``: out is [rows, heads * kv_heads * vdim], every head's weights with the values of every
    KV head (not for one-row segments in BF16)."""
    a = _paged_args(q, k_cache, v_cache, block_table, out, seg, heads, block_size, window, scale, softcap, out_scale, gate, vdim,
                    keep_first, sink, chunk, bias, all_values)
    if q.dtype == torch.float32:
        K._check(K.lib().nx_paged_window_f32(C.byref(a), K._stream()), "nx_paged_window_f32")
    elif seg.max_len == 1 and not all_values:
        a.splits = splits
        if splits > 1:
            a.part_o = K.scratch(seg.count * heads * splits * a.vdim * 4, "window_o", q.device).data_ptr()
            a.part_ml = K.scratch(seg.count * heads * splits * 8, "window_ml", q.device).data_ptr()
        K._check(K.lib().nx_paged_window_decode(C.byref(a), K._stream()), "nx_paged_window_decode")
    else:
        K._check(K.lib().nx_paged_window_prefill(C.byref(a), K._stream()), "nx_paged_window_prefill")


def talk_paged(q, k_cache, v_cache, block_table, out, talk, seg: Segments, *, heads, block_size, window, scale, keys, softcap=0.0,
               splits=1, gate=None, keep_first=0, chunk=0, bias=None) -> None:
    """One-row and short segments of heads that mix their weights (``talk``: FP32 [heads, heads], to, from); ``keys``: the most keys a
    row can see.  The segments run in portions whose scratch stays below `TALK_SCRATCH`."""
    G, Dv, lib = k_cache.shape[2], v_cache.shape[3], K.lib()
    pitch = (keys + min(seg.max_len, 64) + 63) // 64 * 64       # the rows of one tile, up to 64 tokens, see this many together
    each = heads * (pitch * 6 + splits * (8 + (Dv * 4 if splits > 1 else 0)))
    rows = lib.nx_talk_rows(C.c_int(heads), C.c_int(G), C.c_int(seg.count), C.c_int(seg.max_len), C.c_int(seg.total))
    at = max(1, seg.count * TALK_SCRATCH // max(1, rows * each)) if rows * each > TALK_SCRATCH else seg.count
    for i in range(0, seg.count, at):
        part = seg if at >= seg.count else Segments(seg.table, seg.first + i, min(at, seg.count - i), seg.max_len,
                                                    min(seg.total, min(at, seg.count - i) * seg.max_len))
        n = lib.nx_talk_rows(C.c_int(heads), C.c_int(G), C.c_int(part.count), C.c_int(part.max_len), C.c_int(part.total))
        a = TalkPagedArgs(_paged_args(q, k_cache, v_cache, block_table, out, part, heads, block_size, window, scale, softcap, 1.0, gate, 0,
                                      keep_first, None, chunk, bias, False), _ptr(talk), None, None, pitch, n)
        a.base.splits = splits
        a.base.part_ml = K.scratch(n * heads * splits * 8, "window_ml", q.device).data_ptr()
        if splits > 1:
            a.base.part_o = K.scratch(n * heads * splits * Dv * 4, "window_o", q.device).data_ptr()
        a.scores = K.scratch(n * heads * pitch * 4, "talk_scores", q.device).data_ptr()
        a.weights = K.scratch(n * heads * pitch * 2, "talk_weights", q.device).data_ptr()
        K._check(lib.nx_talk_paged(C.byref(a), K._stream()), "nx_talk_paged")


def latent_attention(q, cache, block_table, out, seg: Segments, *, heads, rank, window, scale, gate=None, splits=1) -> None:
    """q: BF16 [rows, heads * row]; cache [blocks, block_size, 1, row], the values are its leading ``rank`` columns; out
    [rows, heads * rank]; ``splits`` spans of the keys run at the same time."""
    a = LatentAttnArgs(_ptr(q), _ptr(cache), _ptr(block_table), _ptr(out), _ptr(gate), None, None,
                       K.status_word(q.device).data_ptr(), q.stride(0), out.stride(0), heads, cache.shape[-1], rank, cache.shape[1],
                       block_table.shape[1], window, splits, cache.shape[0] * cache.shape[1], scale, seg.args())
    if splits > 1:
        n = q.shape[0] * heads * splits
        a.part_o = K.scratch(n * rank * 4, "latent_o", q.device).data_ptr()
        a.part_ml = K.scratch(n * 8, "latent_ml", q.device).data_ptr()
    K._check(K.lib().nx_latent_attention(C.byref(a), K._stream()), "nx_latent_attention")


def latent_prompt(q, kv, lat, out, blocks, *, heads, dim, rot, vdim, rank, window, scale, gate=None) -> None:
    """The same attention on formed keys and values (tcgen05).  q [rows, heads * (dim + rot)], kv [kv rows, heads * (dim + vdim)],
    lat [kv rows, row]: the shared key part at column ``rank``; blocks int32 [n, 4] of up to 256 query rows: first row, rows,
    position of the first row, kv row of position 0."""
    a = LatentPromptArgs(_ptr(q), _ptr(kv), _ptr(lat), _ptr(out), _ptr(gate), _ptr(blocks), K.status_word(q.device).data_ptr(),
                         q.stride(0), kv.stride(0), lat.stride(0), out.stride(0), blocks.shape[0], q.shape[0], kv.shape[0], dim + rot,
                         rank, heads, dim, rot, vdim, window, scale)
    K._check(K.lib().nx_latent_prompt(C.byref(a), K._stream()), "nx_latent_prompt")


def window_prompt(q, k, v, out, blocks, *, heads, kv_heads, dim, vdim, window, scale, keep_first=0, kept=None, sink=None, gate=None,
                  chunk=0, bias=None) -> None:
    """The tcgen05 form on plain grouped keys and values.  q [rows, heads * dim], k [kv rows, kv_heads * dim], v [kv rows, kv_heads *
    vdim]; blocks as in `latent_prompt`; kept int32 [n]: the row that position 0 has among the kept first keys (None: the block's);
    chunk and bias as in `paged_window_attention`."""
    a = WindowPromptArgs(_ptr(q), _ptr(k), _ptr(v), _ptr(out), _ptr(sink), _ptr(blocks), _ptr(kept),
                         K.status_word(q.device).data_ptr(), q.stride(0), k.stride(0), v.stride(0), out.stride(0), blocks.shape[0],
                         q.shape[0], k.shape[0], heads, kv_heads, dim, vdim, window, keep_first, scale, _ptr(gate), _ptr(bias),
                         bias.shape[1] if bias is not None else 0, chunk)
    K._check(K.lib().nx_window_prompt(C.byref(a), K._stream()), "nx_window_prompt")


def extended_bias(bias: torch.Tensor) -> torch.Tensor:
    """The biases [heads, distances] in the layout of `talk_prompt`: units of log2, the first and last one repeated on either side, rows
    of whole 16 bytes."""
    n = bias.shape[1]
    at = torch.arange(-BIAS_MARGIN, (n + BIAS_MARGIN + 3) // 4 * 4, device=bias.device).clamp(0, n - 1)
    return (bias.double() * math.log2(math.e)).float()[:, at].contiguous()


def talk_prompt(q, k, v, out, blocks, *, heads, kv_heads, dim, vdim, window, scale, chunk=0, bias=None, distances=0, row0=0) -> None:
    """`window_prompt` for heads that mix: every head's weights with the values of every KV head, out [rows, heads * kv_heads * vdim].
    ``bias``: `extended_bias` of ``distances`` distances; ``row0``: the query row that the first row of ``out`` belongs to."""
    first = out.data_ptr() - row0 * out.stride(0) * out.element_size()
    a = TalkPromptArgs(_ptr(q), _ptr(k), _ptr(v), first, _ptr(bias), _ptr(blocks), K.status_word(q.device).data_ptr(), q.stride(0),
                       k.stride(0), v.stride(0), out.stride(0), blocks.shape[0], q.shape[0], k.shape[0], heads, kv_heads, dim, vdim,
                       window, chunk, distances, bias.shape[1] if bias is not None else 0, scale)
    K._check(K.lib().nx_talk_prompt(C.byref(a), K._stream()), "nx_talk_prompt")


def talk_prompt_mixed(q, k, v, out, slices, talk, gate, *, heads, kv_heads, dim, vdim, **kw) -> None:
    """`talk_prompt` and the mixture of its outputs (`head_mix`), slice by slice; slices: (blocks, first row, rows), the rows of one slice
    at most ``talk_rows``.  Rows of ``out`` that lie in a slice and in none of its blocks get no defined values."""
    cols = heads * kv_heads * vdim
    wide = K.scratch(max((n for _, _, n in slices), default=0) * cols * q.element_size(), "talk_wide", q.device).view(q.dtype)
    for blocks, row0, n in slices:
        part = wide[: n * cols].view(n, cols)
        talk_prompt(q, k, v, part, blocks, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, row0=row0, **kw)
        head_mix(part, talk, None if gate is None else gate[row0: row0 + n], out[row0: row0 + n], heads=heads, kv_heads=kv_heads, vdim=vdim)


def talk_rows(heads: int, kv_heads: int, vdim: int) -> int:
    """Rows of a slice of `talk_prompt_mixed`."""
    return max(256, TALK_WIDE // (heads * kv_heads * vdim * 2))


def latent_gather(cache, block_table, runs, longest, dst) -> None:
    """Cache rows of ``runs`` (int32 [n, 4]: first row of ``dst``, rows, first position, sequence) into ``dst`` [., row]; cache
    [blocks, block_size, 1, row], or keys or values [blocks, block_size, heads, size] whose rows are heads * size wide."""
    K._check(K.lib().nx_latent_gather(K._p(cache), K._p(dst), K._p(block_table), K._p(runs), C.c_int(runs.shape[0]), C.c_int(longest),
                                      C.c_int(block_table.shape[1]), C.c_int(cache.shape[1]), C.c_int(cache.shape[2] * cache.shape[3]),
                                      K._stream()), "nx_latent_gather")
