"""ctypes bindings of the serving form of expert layers (``nx_api_moe.h``): routing by a table (one launch sorts the assignments
of a step for every layer) or by a sigmoid router (per layer), and the products over the sorted rows (tcgen05 grouped GEMM,
few-rows BF16 kernel, FP32)."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import List, Optional, Sequence, Tuple

import torch

from . import _cuda as K
from ._mixers import Glu, glu

MAX_LAYERS = 32       # layers per routing launch
F32_ALIGN = 32        # slots per tile of the FP32 product


class TableRouteLayer(C.Structure):
    _fields_ = [("table", C.c_void_p), ("slots", C.c_void_p), ("rows", C.c_void_p), ("start", C.c_void_p), ("count", C.c_void_p),
                ("groups", C.c_void_p), ("experts", C.c_int32), ("top", C.c_int32), ("max_slots", C.c_int32)]


class TableRouteArgs(C.Structure):
    _fields_ = [("tokens", C.c_void_p), ("n", C.c_int32), ("vocab", C.c_int32), ("layers", C.c_int32), ("align", C.c_int32),
                ("layer", TableRouteLayer * MAX_LAYERS)]


class ExpertGemmArgs(C.Structure):
    _fields_ = [("x", C.c_void_p), ("rows", C.c_void_p), ("w", C.c_void_p), ("out", C.c_void_p), ("start", C.c_void_p),
                ("count", C.c_void_p), ("groups", C.c_void_p), ("ldx", C.c_int64), ("ldw", C.c_int64), ("stride_w", C.c_int64),
                ("ldo", C.c_int64), ("experts", C.c_int32), ("n", C.c_int32), ("k", C.c_int32), ("act", C.c_int32),
                ("tiles", C.c_int32), ("align", C.c_int32), ("group_x", C.c_int64), ("group_out", C.c_int64), ("m", C.c_int32),
                ("gated", C.c_int32), ("glu", Glu)]


class GateRouteArgs(C.Structure):
    _fields_ = [("logits", C.c_void_p), ("correction", C.c_void_p), ("expert", C.c_void_p), ("weight", C.c_void_p), ("slots", C.c_void_p),
                ("rows", C.c_void_p), ("start", C.c_void_p), ("count", C.c_void_p), ("groups", C.c_void_p), ("h", C.c_void_p),
                ("by_slot", C.c_void_p), ("ld", C.c_int64), ("n", C.c_int32), ("experts", C.c_int32), ("top", C.c_int32),
                ("n_groups", C.c_int32), ("keep", C.c_int32), ("align", C.c_int32), ("max_slots", C.c_int32), ("row_bytes", C.c_int32)]


@dataclass
class Route:
    """The sorted assignments of one layer: slots [n, top], rows [max_slots], start / count [experts], groups [tiles]."""
    slots: torch.Tensor
    rows: torch.Tensor
    start: torch.Tensor
    count: torch.Tensor
    groups: torch.Tensor
    align: int
    top: int
    weight: Optional[torch.Tensor] = None      # FP32 [n, top]; None: equal weights

    @property
    def max_slots(self) -> int:
        return self.rows.shape[0]


def table_slots(assignments: int, experts: int, align: int) -> int:
    """Slots that ``assignments`` can take at most: every expert in use leaves up to align - 1 of them empty."""
    return -(-(assignments + min(assignments, experts) * (align - 1)) // align) * align


def table_route(tokens: torch.Tensor, layers: Sequence[Tuple[torch.Tensor, int]], align: int) -> List[Route]:
    """``layers``: (table [vocab, top] int32, experts) of every layer of experts."""
    n, dev, out = tokens.shape[0], tokens.device, []
    sizes = [(t.shape[1], e, table_slots(n * t.shape[1], e, align)) for t, e in layers]
    buf = torch.empty(sum(n * top + cap + 2 * e + cap // align for top, e, cap in sizes), dtype=torch.int32, device=dev)
    at = 0

    def take(k):
        nonlocal at
        at += k
        return buf[at - k: at]
    for top, e, cap in sizes:
        out.append(Route(take(n * top).view(n, top), take(cap), take(e), take(e), take(cap // align), align, top))
    for first in range(0, len(layers), MAX_LAYERS):
        part = layers[first: first + MAX_LAYERS]
        a = TableRouteArgs(tokens.data_ptr(), n, part[0][0].shape[0], len(part), align)
        for i, (table, experts) in enumerate(part):
            r = out[first + i]
            a.layer[i] = TableRouteLayer(table.data_ptr(), r.slots.data_ptr(), r.rows.data_ptr(), r.start.data_ptr(),
                                         r.count.data_ptr(), r.groups.data_ptr(), experts, r.top, r.max_slots)
        K._check(K.lib().nx_moe_table_route(C.byref(a), K._stream()), "nx_moe_table_route")
    return out


def gate_route(logits: torch.Tensor, correction: torch.Tensor, top: int, align: int, *, n_groups: int = 1, keep: int = 1,
               h: Optional[torch.Tensor] = None) -> Tuple[Route, Optional[torch.Tensor]]:
    """Routing of [n, experts] FP32 logits: scores sigmoid(logits), the choice by score + correction among the experts of the
    ``keep`` best of ``n_groups`` groups, weights from the scores of the chosen.  With ``h`` (contiguous rows) the rows come back in
    slot order too."""
    n, E, dev = logits.shape[0], correction.shape[0], logits.device
    cap = table_slots(n * top, E, align)
    buf = torch.empty(2 * n * top + cap + 2 * E + cap // align, dtype=torch.int32, device=dev)
    expert, slots, rows, start, count, groups = buf.split([n * top, n * top, cap, E, E, cap // align])
    weight = torch.empty((n, top), dtype=torch.float32, device=dev)
    by_slot = None
    if h is not None:
        if not h.is_contiguous():
            raise ValueError("gate_route: h must be contiguous")
        by_slot = torch.empty((cap, h.shape[1]), dtype=h.dtype, device=dev)
    a = GateRouteArgs(logits.data_ptr(), correction.data_ptr(), expert.data_ptr(), weight.data_ptr(), slots.data_ptr(), rows.data_ptr(),
                      start.data_ptr(), count.data_ptr(), groups.data_ptr(), h.data_ptr() if h is not None else None,
                      by_slot.data_ptr() if h is not None else None, logits.stride(0), n, E, top, n_groups, keep, align, cap,
                      h.shape[1] * h.element_size() if h is not None else 0)
    K._check(K.lib().nx_moe_gate_route(C.byref(a), K._stream()), "nx_moe_gate_route")
    return Route(slots.view(n, top), rows, start, count, groups, align, top, weight), by_slot


def expert_product(x: torch.Tensor, w: torch.Tensor, route: Route, *, gather: bool, act: Optional[str] = None,
                   gate: Optional[Glu] = None) -> torch.Tensor:
    """out[slot] = act(w[expert] x[row of slot]), w [experts, n, k].  ``gather``: x has the batch's rows, else the slots'.
    ``gate``: the rows of w are turns of eight gates and eight values; out has n / 2 columns.
    The product is chosen by dtype and the alignment of the route: 1 few rows (BF16), 32 FP32, 128 / 256 the tcgen05 GEMM
    (whose x is in slot order)."""
    E, n, k = w.shape
    few = x.dtype == torch.bfloat16 and route.align < 128
    if gate is not None and not few and route.align == 256 and K.gated_gemm_ok(route.max_slots, n):
        out = torch.empty((route.max_slots, n // 2), dtype=x.dtype, device=x.device)
        return K.grouped_gemm(x, w, route.groups, route.align, out=out, glu=gate)
    if gate is not None and not few:
        both = expert_product(x, w, route, gather=gather)
        out = torch.empty((route.max_slots, n // 2), dtype=x.dtype, device=x.device)
        glu(both, out, gate, interleaved=True)
        return out
    if gate is not None:
        n //= 2
    out = torch.empty((route.max_slots, n), dtype=x.dtype, device=x.device)
    if x.dtype == torch.bfloat16 and route.align >= 128:
        if gather:
            raise ValueError("expert_product: the GEMM reads its rows in slot order")
        return K.grouped_gemm(x, w, route.groups, route.align, act=act, out=out)
    a = ExpertGemmArgs(x.data_ptr(), route.rows.data_ptr() if gather else None, w.data_ptr(), out.data_ptr(), route.start.data_ptr(),
                       route.count.data_ptr(), route.groups.data_ptr(), x.stride(0), w.stride(1), w.stride(0), out.stride(0), E,
                       w.shape[1], k, K.ACT[act], route.groups.shape[0], route.align, 0, 0, route.slots.shape[0], int(gate is not None),
                       gate or Glu())
    name = "nx_expert_skinny" if x.dtype == torch.bfloat16 else "nx_expert_f32"
    K._check(getattr(K.lib(), name)(C.byref(a), K._stream()), name)
    return out


def head_product(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
    """out[:, h] = x[:, h] w[h]^T for few rows: x [rows, heads, >= k] and out [rows, heads, >= n] views, w BF16 [heads, n, k]."""
    H, n, k = w.shape
    a = ExpertGemmArgs(x.data_ptr(), None, w.data_ptr(), out.data_ptr(), None, None, None, x.stride(0), w.stride(1), w.stride(0),
                       out.stride(0), H, n, k, K.ACT[None], 0, 1, x.stride(1), out.stride(1), x.shape[0], 0, Glu())
    K._check(K.lib().nx_expert_skinny(C.byref(a), K._stream()), "nx_expert_skinny")
