// Mixture-of-experts routing on the GPU: top-k selection with the gate softmax over the selected
// experts (FP32 router logits in), capacity assignment in priority order (choice j first, then token
// index: a per-expert counting sort, deterministic), and the gate gradient of the combine step.
// Tokens are then gathered into per-expert [capacity, d] buffers and combined by the dispatch / combine
// kernels (which also serve expert parallelism over peer memory); the expert FFN itself is a strided
// batched tcgen05 GEMM over the padded buffers.
// Parity: src/moe/moe.cpp (router, capacity, permutation) of the reference, which runs on the CPU.
// Serving: experts that a table picks by token id need no router, one launch sorts a step's assignments for every layer; a
// sigmoid router with a correction and groups of experts picks and sorts per layer.  The serving forms of the expert products
// (few rows per expert; FP32) live here too.
#include "common.cuh"
#include "mixer_common.cuh"
#include "nx_api_moe.h"

#include <algorithm>

namespace {
using namespace nx;

// warp per token; E <= 1024; k <= 8
__global__ void moe_topk_kernel(const float* __restrict__ logits, int tokens, int E, int k,
                                int32_t* __restrict__ expert, float* __restrict__ gate) {
  const int t = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (t >= tokens) return;
  const float* row = logits + static_cast<int64_t>(t) * E;
  float sel_v[8];
  int sel_i[8];
  for (int j = 0; j < k; ++j) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      bool taken = false;
      for (int q = 0; q < j; ++q) taken |= sel_i[q] == e;
      const float v = row[e];
      if (!taken && (v > best || (v == best && e < bi))) {
        best = v;
        bi = e;
      }
    }
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) {
        best = ov;
        bi = oi;
      }
    }
    sel_v[j] = best;
    sel_i[j] = bi;
  }
  if (lane == 0) {
    float mx = sel_v[0], se = 0.0f;
    for (int j = 0; j < k; ++j) se += expf(sel_v[j] - mx);
    for (int j = 0; j < k; ++j) {
      expert[t * k + j] = sel_i[j];
      gate[t * k + j] = expf(sel_v[j] - mx) / se;
    }
  }
}

// One block per expert.  Entries are visited in priority order p = j * tokens + t; entry (t, j) of this
// expert gets slot = number of earlier entries of the same expert, or -1 beyond the capacity.
__global__ void __launch_bounds__(1024)
moe_assign_kernel(const int32_t* __restrict__ expert, int tokens, int k, int capacity, int32_t* __restrict__ slot,
                  int32_t* __restrict__ counts, int32_t* __restrict__ dropped) {
  __shared__ int s_warp[32];
  __shared__ int s_run;
  const int e = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) s_run = 0;
  __syncthreads();
  const int total = tokens * k;
  int ndrop = 0;
  for (int base = 0; base < total; base += blockDim.x) {
    const int p = base + threadIdx.x;
    int t = 0, j = 0;
    bool mine = false;
    if (p < total) {
      j = p / tokens;
      t = p % tokens;
      mine = expert[t * k + j] == e;
    }
    const unsigned ballot = __ballot_sync(0xffffffffu, mine);
    const int within = __popc(ballot & ((1u << lane) - 1));
    if (lane == 0) s_warp[warp] = __popc(ballot);
    __syncthreads();
    int before = s_run;
    for (int w = 0; w < warp; ++w) before += s_warp[w];
    if (mine) {
      const int s = before + within;
      const bool ok = s < capacity;
      slot[t * k + j] = ok ? s : -1;
      ndrop += ok ? 0 : 1;
    }
    __syncthreads();
    if (threadIdx.x == 0) {
      int sum = 0;
      for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) sum += s_warp[w];
      s_run += sum;
    }
    __syncthreads();
  }
  if (threadIdx.x == 0) counts[e] = min(s_run, capacity);
  if (dropped != nullptr && ndrop > 0) atomicAdd(dropped, ndrop);
}

// Capacity per GROUP of tokens and the Reroute overflow policy.  One warp per group walks the group's assignments in
// priority order (choice j, then token t) with the per-expert fill counters in shared memory: an assignment whose
// expert is full is dropped (slot -1) or, with `order` given ([tokens, E]: every token's experts by descending
// score), moved to the token's best expert that still has room and is not one of the token's own choices; the lanes
// test 32 candidates per trip.  slot = group * capacity + position inside the group's share of the expert's buffer,
// so the buffers are [E, groups * capacity, d].  counts[g * E + e] = rows of group g accepted by expert e.
__global__ void __launch_bounds__(32)
moe_assign_groups_kernel(int32_t* __restrict__ expert, const int32_t* __restrict__ order, int tokens, int k, int E,
                         int groups, int capacity, int32_t* __restrict__ slot, int32_t* __restrict__ counts,
                         int32_t* __restrict__ dropped, int32_t* __restrict__ rerouted) {
  extern __shared__ int s_fill[];  // [E]
  const int g = blockIdx.x, lane = threadIdx.x;
  const int ng = tokens / groups, t0 = g * ng;
  for (int e = lane; e < E; e += 32) s_fill[e] = 0;
  __syncwarp();
  int ndrop = 0, nmove = 0;
  for (int j = 0; j < k; ++j) {
    for (int t = t0; t < t0 + ng; ++t) {
      int e = expert[t * k + j];
      bool full = s_fill[e] >= capacity;
      if (full && order != nullptr) {
        int alt = -1;
        for (int c0 = 0; c0 < E && alt < 0; c0 += 32) {
          const int c = c0 + lane;
          bool ok = false;
          int cand = -1;
          if (c < E) {
            cand = order[static_cast<int64_t>(t) * E + c];
            ok = s_fill[cand] < capacity;
            for (int q = 0; q < k; ++q) ok = ok && expert[t * k + q] != cand;
          }
          const unsigned b = __ballot_sync(0xffffffffu, ok);
          if (b != 0u) alt = __shfl_sync(0xffffffffu, cand, __ffs(b) - 1);
        }
        if (alt >= 0) {
          e = alt;
          full = false;
          ++nmove;
          if (lane == 0) expert[t * k + j] = e;
        }
      }
      if (lane == 0) {
        slot[t * k + j] = full ? -1 : g * capacity + s_fill[e];
        if (!full) s_fill[e] += 1;
      }
      ndrop += full ? 1 : 0;
      __syncwarp();
    }
  }
  for (int e = lane; e < E; e += 32) counts[g * E + e] = s_fill[e];
  if (lane == 0) {
    if (dropped != nullptr && ndrop > 0) atomicAdd(dropped, ndrop);
    if (rerouted != nullptr && nmove > 0) atomicAdd(rerouted, nmove);
  }
}

// dgate[t, j] = dy[t] . expert_out[e_tj][slot_tj]   (0 for dropped assignments); warp per (t, j)
__global__ void moe_gate_grad_kernel(const __nv_bfloat16* __restrict__ dy, const __nv_bfloat16* __restrict__ buf,
                                     const int32_t* __restrict__ expert, const int32_t* __restrict__ slot,
                                     float* __restrict__ dgate, int entries, int k, int d, int capacity) {
  const int i = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  if (i >= entries) return;
  const int s = slot[i];
  float acc = 0.0f;
  if (s >= 0) {
    const __nv_bfloat16* a = dy + static_cast<int64_t>(i / k) * d;
    const __nv_bfloat16* b = buf + (static_cast<int64_t>(expert[i]) * capacity + s) * d;
    for (int c = lane * 2; c < d; c += 64) {
      const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(a + c);
      const __nv_bfloat162 y = *reinterpret_cast<const __nv_bfloat162*>(b + c);
      acc += __low2float(x) * __low2float(y) + __high2float(x) * __high2float(y);
    }
  }
  acc = warp_sum(acc);
  if (lane == 0) dgate[i] = acc;
}

// ------------------------------------------------------------------------------------------------
// experts by token id: one block per layer counts, places and scatters its assignments
// ------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(1024) moe_table_route_kernel(const __grid_constant__ NxTableRouteArgs a) {
  extern __shared__ int s_cnt[];               // [experts] counts, then the next free slot
  __shared__ int s_warp[32], s_total;
  const NxTableRouteLayer& L = a.layer[blockIdx.x];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  for (int e = tid; e < L.experts; e += blockDim.x) s_cnt[e] = 0;
  for (int i = tid; i < L.max_slots; i += blockDim.x) L.rows[i] = -1;
  __syncthreads();
#pragma unroll 4
  for (int r = tid; r < a.n; r += blockDim.x) {
    const int t = a.tokens[r];
    const int32_t* row = L.table + static_cast<int64_t>(t >= 0 && t < a.vocab ? t : 0) * L.top;
    for (int j = 0; j < L.top; ++j) {
      const int e = row[j];
      L.slots[r * L.top + j] = e;              // the expert for now, read again by this thread
      atomicAdd(&s_cnt[e], 1);
    }
  }
  __syncthreads();
  int base = 0;
  for (int e0 = 0; e0 < L.experts; e0 += blockDim.x) {
    const int e = e0 + tid, n = e < L.experts ? s_cnt[e] : 0, padded = (n + a.align - 1) / a.align * a.align;
    int incl = padded;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += v;
    }
    if (lane == 31) s_warp[warp] = incl;
    __syncthreads();
    int before = base;
    for (int w = 0; w < warp; ++w) before += s_warp[w];
    const int first = before + incl - padded;
    if (e < L.experts) {
      L.start[e] = first;
      L.count[e] = n;
      s_cnt[e] = first;
      for (int g = first / a.align; g < (first + padded) / a.align; ++g) L.groups[g] = e;
    }
    if (tid == static_cast<int>(blockDim.x) - 1) s_total = before + incl;
    __syncthreads();
    base = s_total;
  }
  for (int g = base / a.align + tid; g < L.max_slots / a.align; g += blockDim.x) L.groups[g] = -1;
#pragma unroll 4
  for (int r = tid; r < a.n; r += blockDim.x)
    for (int j = 0; j < L.top; ++j) {
      const int s = atomicAdd(&s_cnt[L.slots[r * L.top + j]], 1);
      L.slots[r * L.top + j] = s;
      L.rows[s] = r;
    }
}

// ------------------------------------------------------------------------------------------------
// experts by a sigmoid router
// ------------------------------------------------------------------------------------------------
// One warp picks the experts of one row: lane j < top returns the j-th expert and its weight.  s: 2 * experts floats of the warp.
__device__ __forceinline__ void pick_experts(const NxGateRouteArgs& a, int row, float* s, int& expert, float& weight) {
  const int lane = threadIdx.x & 31, E = a.experts;
  const float* z = a.logits + row * a.ld;
  float* g = s + E;
  __syncwarp();
  for (int e = lane; e < E; e += 32) s[e] = sigmoid_exact(z[e]) + a.correction[e];
  __syncwarp();
  if (a.n_groups > 1 && a.keep < a.n_groups) {
    const int size = E / a.n_groups;
    for (int i = lane; i < a.n_groups; i += 32) {
      float first = -INFINITY, second = -INFINITY;
      for (int e = i * size; e < (i + 1) * size; ++e) {
        second = fmaxf(second, fminf(first, s[e]));
        first = fmaxf(first, s[e]);
      }
      g[i] = size > 1 ? first + second : first;
    }
    __syncwarp();
    for (int i = lane; i < a.n_groups; i += 32) {
      int better = 0;
      for (int o = 0; o < a.n_groups; ++o) better += g[o] > g[i] || (g[o] == g[i] && o < i) ? 1 : 0;
      if (better >= a.keep)
        for (int e = i * size; e < (i + 1) * size; ++e) s[e] = -INFINITY;
    }
    __syncwarp();
  }
  int mine = 0;
  for (int j = 0; j < a.top; ++j) {
    float best = -INFINITY;
    int be = 0x7fffffff;
    for (int e = lane; e < E; e += 32)
      if (s[e] > best) {
        best = s[e];
        be = e;
      }
    const int bits = __float_as_int(best), key = bits < 0 ? bits ^ 0x7fffffff : bits;     // ordered like the floats
    const int top_key = __reduce_max_sync(0xffffffffu, key);
    be = __reduce_min_sync(0xffffffffu, key == top_key ? be : 0x7fffffff);
    if (be >= E) be = j;                       // only where scores are not numbers
    if (lane == j) mine = be;
    if (lane == (be & 31)) s[be] = -INFINITY;
    __syncwarp();
  }
  const float w = lane < a.top ? sigmoid_exact(z[mine]) : 0.0f;
  expert = mine;
  weight = w / (warp_sum(w) + 1e-20f);
}

// first[e] = slots before expert e, every expert's share rounded up to `align`; returns the total.  All threads of the block.
__device__ int expert_starts(const int32_t* count, int experts, int align, int* first) {
  __shared__ int s_warp[32], s_total;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  int base = 0;
  for (int e0 = 0; e0 < experts; e0 += blockDim.x) {
    const int e = e0 + tid, padded = e < experts ? (count[e] + align - 1) / align * align : 0;
    int incl = padded;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += v;
    }
    if (lane == 31) s_warp[warp] = incl;
    __syncthreads();
    int before = base;
    for (int w = 0; w < warp; ++w) before += s_warp[w];
    if (e < experts) first[e] = before + incl - padded;
    if (tid == static_cast<int>(blockDim.x) - 1) s_total = before + incl;
    __syncthreads();
    base = s_total;
  }
  return base;
}
// start, groups and the empty slots, by the threads of one block
__device__ void expert_tables(const NxGateRouteArgs& a, const int32_t* count, const int* first, int total) {
  for (int e = threadIdx.x; e < a.experts; e += blockDim.x) {
    const int n = count[e], padded = (n + a.align - 1) / a.align * a.align;
    a.start[e] = first[e];
    for (int i = first[e] / a.align; i < (first[e] + padded) / a.align; ++i) a.groups[i] = e;
    for (int i = first[e] + n; i < first[e] + padded; ++i) a.rows[i] = -1;
  }
  for (int i = total / a.align + threadIdx.x; i < a.max_slots / a.align; i += blockDim.x) a.groups[i] = -1;
  for (int i = total + threadIdx.x; i < a.max_slots; i += blockDim.x) a.rows[i] = -1;
}

// few rows: everything in one block
__global__ void __launch_bounds__(1024) gate_route_small_kernel(const NxGateRouteArgs a) {
  extern __shared__ float s_score[];           // [warps][2 * experts], then int [2 * experts]: counts, starts
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5, E = a.experts;
  int* s_cnt = reinterpret_cast<int*>(s_score + warps * 2 * E);
  int* s_first = s_cnt + E;
  for (int e = threadIdx.x; e < E; e += blockDim.x) s_cnt[e] = 0;
  __syncthreads();
  for (int r = warp; r < a.n; r += warps) {
    int e;
    float w;
    pick_experts(a, r, s_score + warp * 2 * E, e, w);
    if (lane < a.top) {
      a.expert[r * a.top + lane] = e;
      a.weight[r * a.top + lane] = w;
      a.slots[r * a.top + lane] = atomicAdd(&s_cnt[e], 1);     // place inside the expert; read again by this thread
    }
  }
  __syncthreads();
  const int total = expert_starts(s_cnt, E, a.align, s_first);
  __syncthreads();
  expert_tables(a, s_cnt, s_first, total);
  for (int e = threadIdx.x; e < E; e += blockDim.x) a.count[e] = s_cnt[e];
  for (int r = warp; r < a.n; r += warps)
    if (lane < a.top) {
      const int s = s_first[a.expert[r * a.top + lane]] + a.slots[r * a.top + lane];
      a.slots[r * a.top + lane] = s;
      a.rows[s] = r;
    }
}

constexpr int kPickRows = 32;                  // rows per block, 8 warps
__global__ void __launch_bounds__(256) gate_pick_kernel(const NxGateRouteArgs a) {
  extern __shared__ float s_score[];           // [8][2 * experts], then int [experts]: counts, then the block's first places
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, E = a.experts;
  int* s_cnt = reinterpret_cast<int*>(s_score + 8 * 2 * E);
  for (int e = threadIdx.x; e < E; e += 256) s_cnt[e] = 0;
  __syncthreads();
  int expert[kPickRows / 8], place[kPickRows / 8];
#pragma unroll
  for (int i = 0; i < kPickRows / 8; ++i) {
    const int r = blockIdx.x * kPickRows + i * 8 + warp;
    expert[i] = -1;
    if (r >= a.n) continue;
    float w;
    pick_experts(a, r, s_score + warp * 2 * E, expert[i], w);
    if (lane < a.top) {
      a.expert[r * a.top + lane] = expert[i];
      a.weight[r * a.top + lane] = w;
      place[i] = atomicAdd(&s_cnt[expert[i]], 1);
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += 256) {
    const int n = s_cnt[e];
    s_cnt[e] = n > 0 ? atomicAdd(&a.count[e], n) : 0;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < kPickRows / 8; ++i) {
    const int r = blockIdx.x * kPickRows + i * 8 + warp;
    if (expert[i] >= 0 && lane < a.top) a.slots[r * a.top + lane] = s_cnt[expert[i]] + place[i];
  }
}

// a warp per row: places inside experts become slots, the row is copied to them; block 0 writes the tables
__global__ void __launch_bounds__(256) gate_place_kernel(const NxGateRouteArgs a) {
  extern __shared__ int s_first[];
  const int total = expert_starts(a.count, a.experts, a.align, s_first);
  __syncthreads();
  if (blockIdx.x == 0) expert_tables(a, a.count, s_first, total);
  const int lane = threadIdx.x & 31, chunks = a.row_bytes / 16;
  for (int r = blockIdx.x * 8 + (threadIdx.x >> 5); r < a.n; r += gridDim.x * 8) {
    int slot = 0;
    if (lane < a.top) {
      slot = s_first[a.expert[r * a.top + lane]] + a.slots[r * a.top + lane];
      a.slots[r * a.top + lane] = slot;
      a.rows[slot] = r;
    }
    if (a.by_slot == nullptr) continue;
    const uint4* src = static_cast<const uint4*>(a.h) + static_cast<int64_t>(r) * chunks;
    for (int c0 = 0; c0 < chunks; c0 += 128) {
      uint4 v[4];
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (c0 + u * 32 + lane < chunks) v[u] = __ldg(src + c0 + u * 32 + lane);
      for (int j = 0; j < a.top; ++j) {
        uint4* dst = static_cast<uint4*>(a.by_slot) + static_cast<int64_t>(__shfl_sync(0xffffffffu, slot, j)) * chunks;
#pragma unroll
        for (int u = 0; u < 4; ++u)
          if (c0 + u * 32 + lane < chunks) dst[c0 + u * 32 + lane] = v[u];
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------
// product with one weight matrix per group (expert, head), few rows: the weights stream through registers once for up to
// 8 NT rows.  A thread's 16-byte load covers eight neighbours along K; the sum over K may take them in any order as long as
// both operands agree, so each load is two k-steps of the tensor-core tile as it is.  A block has four warps: 4 / KS tiles of
// 16 weight rows, each cut into KS parts along K whose sums meet in shared memory.
// ------------------------------------------------------------------------------------------------
template <int NT, int KS>
__device__ __forceinline__ void group_rows(const NxExpertGemmArgs& a, int group, int tile, int first, int cnt, float* s_acc) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int part = warp % KS, n0 = (tile * (4 / KS) + warp / KS) * 16;
  const int k_part = ((a.k + KS - 1) / KS + 63) / 64 * 64, k_end = min(a.k, (part + 1) * k_part);
  const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(a.w) + group * a.stride_w;
  const __nv_bfloat16 *w0 = w + static_cast<int64_t>(n0 + g) * a.ldw + t * 8, *w1 = w0 + 8 * a.ldw;
  const bool in0 = n0 + g < a.n, in1 = n0 + g + 8 < a.n;
  const __nv_bfloat16* x[NT];
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    const int s = first + min(i * 8 + g, cnt - 1);           // rows past the last repeat it; they are not stored
    x[i] = static_cast<const __nv_bfloat16*>(a.x) + group * a.group_x +
           static_cast<int64_t>(a.rows != nullptr ? a.rows[s] : s) * a.ldx + t * 8;
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.0f;
  }
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll(NT <= 2 ? 4 : 2)
  for (int k0 = part * k_part; k0 < k_end; k0 += 64) {
    uint4 wa[2], wb[2], v[NT][2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const bool ink = k0 + h * 32 + t * 8 < k_end;
      wa[h] = ink && in0 ? __ldcs(reinterpret_cast<const uint4*>(w0 + k0 + h * 32)) : zero;
      wb[h] = ink && in1 ? __ldcs(reinterpret_cast<const uint4*>(w1 + k0 + h * 32)) : zero;
#pragma unroll
      for (int i = 0; i < NT; ++i) v[i][h] = ink ? __ldg(reinterpret_cast<const uint4*>(x[i] + k0 + h * 32)) : zero;
    }
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const uint32_t f0[4] = {wa[h].x, wb[h].x, wa[h].y, wb[h].y}, f1[4] = {wa[h].z, wb[h].z, wa[h].w, wb[h].w};
        mma_bf16(acc[i], f0, v[i][h].x, v[i][h].y);
        mma_bf16(acc[i], f1, v[i][h].z, v[i][h].w);
      }
  }
  if constexpr (KS > 1) {
    __syncthreads();                                         // a previous round has read s_acc
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) s_acc[(warp * NT * 4 + i * 4 + e) * 32 + lane] = acc[i][e];
    __syncthreads();
    if (part != 0) return;
#pragma unroll
    for (int p = 1; p < KS; ++p)
#pragma unroll
      for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] += s_acc[((warp + p) * NT * 4 + i * 4 + e) * 32 + lane];
  }
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + group * a.group_out;
  if (a.gated) {                       // the tile's rows are eight gates and the eight values that belong to them
    if (!in1) return;
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int s = i * 8 + t * 2 + e;
        if (s < cnt)
          out[static_cast<int64_t>(first + s) * a.ldo + n0 / 2 + g] = __float2bfloat16_rn(glu_apply<false>(a.glu, acc[i][e], acc[i][e + 2]));
      }
    return;
  }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int s = i * 8 + t * 2 + (e & 1), n = n0 + g + (e >> 1) * 8;
      float v = acc[i][e];
      if (a.act == NX_ACT_RELU2) v = fmaxf(v, 0.0f) * fmaxf(v, 0.0f);
      if (s < cnt && n < a.n) out[static_cast<int64_t>(first + s) * a.ldo + n] = __float2bfloat16_rn(v);
    }
}

template <int KS>
__global__ void __launch_bounds__(128) expert_skinny_kernel(const NxExpertGemmArgs a) {
  __shared__ float s_acc[KS > 1 ? 4 * 4 * 4 * 32 : 1];
  const int group = blockIdx.y, step = 32 * gridDim.z;
  const int all = a.count != nullptr ? a.count[group] : a.m, start = a.start != nullptr ? a.start[group] : 0;
  for (int c0 = blockIdx.z * 32; c0 < all; c0 += step) {     // the same for the whole block
    const int cnt = min(32, all - c0);
    if (cnt <= 8) group_rows<1, KS>(a, group, blockIdx.x, start + c0, cnt, s_acc);
    else if (cnt <= 16) group_rows<2, KS>(a, group, blockIdx.x, start + c0, cnt, s_acc);
    else group_rows<4, KS>(a, group, blockIdx.x, start + c0, cnt, s_acc);
  }
}

// FP32: 32 slots x 64 columns per block, 16 x 16 threads of 2 x 4
__global__ void __launch_bounds__(256) expert_f32_kernel(const NxExpertGemmArgs a) {
  __shared__ float s_x[16][33], s_w[16][65];
  const int e = a.groups[blockIdx.y];
  if (e < 0) return;
  const int s0 = blockIdx.y * 32, n0 = blockIdx.x * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const float *x = static_cast<const float*>(a.x), *w = static_cast<const float*>(a.w) + static_cast<int64_t>(e) * a.stride_w;
  const int last = a.start[e] + a.count[e];
  float acc[2][4] = {{0.0f, 0.0f, 0.0f, 0.0f}, {0.0f, 0.0f, 0.0f, 0.0f}};
  for (int k0 = 0; k0 < a.k; k0 += 16) {
    for (int i = threadIdx.x; i < 32 * 16; i += 256) {
      const int s = s0 + i / 16, k = k0 + i % 16;
      const bool in = s < last && k < a.k;
      const int64_t row = in ? (a.rows != nullptr ? a.rows[s] : s) : 0;
      s_x[i % 16][i / 16] = in ? x[row * a.ldx + k] : 0.0f;
    }
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int n = n0 + i / 16, k = k0 + i % 16;
      s_w[i % 16][i / 16] = n < a.n && k < a.k ? w[static_cast<int64_t>(n) * a.ldw + k] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k)
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(s_x[k][ty * 2 + i], s_w[k][tx * 4 + j], acc[i][j]);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int s = s0 + ty * 2 + i, n = n0 + tx * 4 + j;
      float v = acc[i][j];
      if (a.act == NX_ACT_RELU2) v = fmaxf(v, 0.0f) * fmaxf(v, 0.0f);
      if (s < last && n < a.n) static_cast<float*>(a.out)[static_cast<int64_t>(s) * a.ldo + n] = v;
    }
}

int check_expert(const NxExpertGemmArgs* a) {
  if (a == nullptr || a->x == nullptr || a->w == nullptr || a->out == nullptr || (a->start == nullptr) != (a->count == nullptr)) return -1;
  if (a->experts <= 0 || a->n <= 0 || a->k <= 0 || (a->act != NX_ACT_NONE && a->act != NX_ACT_RELU2)) return -1;
  if (a->gated && ((a->n & 15) || a->act != NX_ACT_NONE)) return -1;
  return 0;
}
}  // namespace

extern "C" int nx_moe_table_route(const NxTableRouteArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->layers < 0 || a->layers > NX_TABLE_LAYERS || a->align < 1 || a->vocab < 1) return -1;
  if (a->layers == 0 || a->n <= 0) return 0;
  int most = 0;
  for (int l = 0; l < a->layers; ++l) {
    const NxTableRouteLayer& L = a->layer[l];
    if (L.experts < 1 || L.experts > 8192 || L.top < 1 || L.max_slots % a->align) return -1;
    // every expert that is used leaves fewer than `align` slots empty
    const int64_t total = static_cast<int64_t>(a->n) * L.top, used = total < L.experts ? total : L.experts;
    if ((total + used * (a->align - 1)) / a->align * a->align > L.max_slots) return -1;
    most = most > L.experts ? most : L.experts;
  }
  moe_table_route_kernel<<<a->layers, 1024, most * sizeof(int), static_cast<cudaStream_t>(stream)>>>(*a);
  return launch_status();
}

extern "C" int nx_moe_gate_route(const NxGateRouteArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->align < 1 || a->experts < 1 || a->experts > 1024 || a->top < 1 || a->top > 32 || a->top > a->experts) return -1;
  if (a->n_groups < 1 || a->experts % a->n_groups || a->keep < 1 || a->keep > a->n_groups || a->max_slots % a->align) return -1;
  if (a->keep * (a->experts / a->n_groups) < a->top || a->ld < a->experts) return -1;
  if (a->by_slot != nullptr && (a->h == nullptr || a->row_bytes <= 0 || (a->row_bytes & 15) ||
                                ((reinterpret_cast<uintptr_t>(a->h) | reinterpret_cast<uintptr_t>(a->by_slot)) & 15)))
    return -1;
  if (a->n <= 0) return 0;
  const int64_t assignments = static_cast<int64_t>(a->n) * a->top, used = assignments < a->experts ? assignments : a->experts;
  if ((assignments + used * (a->align - 1)) / a->align * a->align > a->max_slots) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int E = a->experts;
  if (a->n <= 256 && a->by_slot == nullptr) {
    const int warps = std::max(4, std::min({32, (a->n + 1) / 2, 64 * 1024 / (E * 8)}));
    const int smem = (warps + 1) * 2 * E * 4;
    if (smem > 48 * 1024 && cudaFuncSetAttribute(gate_route_small_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024) != cudaSuccess)
      return -2;
    gate_route_small_kernel<<<1, warps * 32, smem, st>>>(*a);
    return launch_status();
  }
  const int smem = 17 * E * 4;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(gate_pick_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024) != cudaSuccess)
    return -2;
  if (cudaMemsetAsync(a->count, 0, sizeof(int32_t) * E, st) != cudaSuccess) return -2;
  gate_pick_kernel<<<(a->n + kPickRows - 1) / kPickRows, 256, smem, st>>>(*a);
  gate_place_kernel<<<std::min((a->n + 7) / 8, 1184), 256, E * sizeof(int), st>>>(*a);
  return launch_status();
}

extern "C" int nx_expert_skinny(const NxExpertGemmArgs* a, nx_stream_t stream) {
  if (check_expert(a) || (a->k & 7) || (a->ldx & 7) || (a->ldw & 7) || (a->stride_w & 7) || (a->group_x & 7) || a->experts > 65535)
    return -1;
  if ((reinterpret_cast<uintptr_t>(a->x) & 15) || (reinterpret_cast<uintptr_t>(a->w) & 15)) return -1;
  if (a->m <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  // a token uses an expert at most once, so no group has more than m rows
  const int rounds = std::min((a->m + 31) / 32, 8), ks = a->k >= 1024 ? 4 : a->k >= 256 ? 2 : 1, per = 64 / ks;
  const dim3 grid((a->n + per - 1) / per, a->experts, rounds);
  if (ks == 4) expert_skinny_kernel<4><<<grid, 128, 0, st>>>(*a);
  else if (ks == 2) expert_skinny_kernel<2><<<grid, 128, 0, st>>>(*a);
  else expert_skinny_kernel<1><<<grid, 128, 0, st>>>(*a);
  return launch_status();
}

extern "C" int nx_expert_f32(const NxExpertGemmArgs* a, nx_stream_t stream) {
  if (check_expert(a) || a->start == nullptr || a->groups == nullptr || a->align != 32 || a->tiles < 0 || a->tiles > 65535 || a->gated) return -1;
  if (a->tiles == 0) return 0;
  expert_f32_kernel<<<dim3((a->n + 63) / 64, a->tiles), 256, 0, static_cast<cudaStream_t>(stream)>>>(*a);
  return launch_status();
}

extern "C" int nx_moe_topk(const float* logits, int tokens, int experts, int k, int32_t* expert, float* gate,
                           nx_stream_t stream) {
  if (tokens <= 0) return 0;
  if (k < 1 || k > 8 || k > experts || experts > 1024) return -1;
  moe_topk_kernel<<<(tokens + 7) / 8, 256, 0, static_cast<cudaStream_t>(stream)>>>(logits, tokens, experts, k, expert, gate);
  return launch_status();
}

extern "C" int nx_moe_assign(const int32_t* expert, int tokens, int k, int experts, int capacity, int32_t* slot,
                             int32_t* counts, int32_t* dropped, nx_stream_t stream) {
  if (tokens <= 0 || experts <= 0) return 0;
  if (capacity < 0) return -1;
  moe_assign_kernel<<<experts, 1024, 0, static_cast<cudaStream_t>(stream)>>>(expert, tokens, k, capacity, slot, counts, dropped);
  return launch_status();
}

extern "C" int nx_moe_assign_groups(int32_t* expert, const int32_t* order, int tokens, int k, int experts, int groups,
                                    int capacity, int32_t* slot, int32_t* counts, int32_t* dropped, int32_t* rerouted,
                                    nx_stream_t stream) {
  if (tokens <= 0 || experts <= 0) return 0;
  if (groups < 1 || tokens % groups || capacity < 0 || k < 1 || k > 8 || experts > 8192) return -1;
  moe_assign_groups_kernel<<<groups, 32, experts * sizeof(int), static_cast<cudaStream_t>(stream)>>>(
      expert, order, tokens, k, experts, groups, capacity, slot, counts, dropped, rerouted);
  return launch_status();
}

extern "C" int nx_moe_gate_grad(const void* dy, const void* expert_out, const int32_t* expert, const int32_t* slot,
                                float* dgate, int tokens, int k, int d, int capacity, nx_stream_t stream) {
  const int entries = tokens * k;
  if (entries <= 0) return 0;
  if (d & 1) return -1;
  moe_gate_grad_kernel<<<(entries + 7) / 8, 256, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const __nv_bfloat16*>(dy), static_cast<const __nv_bfloat16*>(expert_out), expert, slot, dgate, entries,
      k, d, capacity);
  return launch_status();
}
