// What the paged attention kernels of any head sizes share: the map from products to scores, the keys a block meets, and their rows
// in the cache.
#pragma once
#include "mixer_common.cuh"
#include "nx_api_mixers.h"
#include "paged_common.cuh"

namespace nx {

constexpr float kLog2e = 1.4426950408889634f;

// Scores in units of log2.  Soft-capping goes through one exponential: cap tanh(z) = cap - 2 cap / (1 + e^{2z}).  It is
// monotone, so row maxima are taken over the raw products and only the maximum is mapped.
struct ScoreMap {
  bool capped;
  float mul, cap2, cap;      // capped: x -> cap - cap2 / (1 + 2^(mul x)); else x -> mul x
  __device__ __forceinline__ ScoreMap(float scale, float softcap) {
    capped = softcap > 0.0f;
    mul = capped ? 2.0f * kLog2e * scale / softcap : scale * kLog2e;
    cap = softcap * kLog2e;
    cap2 = 2.0f * cap;
  }
  __device__ __forceinline__ float operator()(float x) const {       // -inf (nothing visible) stays -inf
    if (!capped || x == -INFINITY) return mul * x;
    return cap - cap2 * rcp_approx(1.0f + ex2_approx(mul * x));
  }
  // 2^(mapped x - base)
  __device__ __forceinline__ float prob(float x, float base) const {
    if (!capped) return ex2_approx(fmaf(mul, x, -base));
    return ex2_approx(fmaf(-cap2, rcp_approx(1.0f + ex2_approx(mul * x)), cap - base));
  }
};

// the first key a row at position p sees, apart from the kept first ones
__device__ __forceinline__ int first_key(const NxPagedWindowArgs& a, int p) {
  const int lo = a.window > 0 ? max(0, p - a.window + 1) : 0;
  return a.chunk > 0 ? max(lo, p / a.chunk * a.chunk) : lo;
}

// The keys a block meets, numbered without the gap between the kept first ones and the window: index i is position i below
// `kept` and position i + skip from there on.
struct KeyRange {
  int kept, skip, count;
  // rows at positions pos .. last
  __device__ __forceinline__ KeyRange(const NxPagedWindowArgs& a, int pos, int last) {
    const int lo = first_key(a, pos);
    kept = min(a.keep_first, lo);
    skip = lo - kept;
    count = last + 1 - skip;
  }
  __device__ __forceinline__ int position(int i) const { return i < kept ? i : i + skip; }
};

// the rows of one sequence's keys and values of one KV head each
struct KvSource {
  const __nv_bfloat16 *k, *v;
  const int32_t* bt;
  int64_t k_pitch, v_pitch;                            // elements between cache slots
  int block_size, shift, dim, vdim;                    // shift: log2 of a power-of-two block size, else -1
  __device__ __forceinline__ KvSource(const NxPagedWindowArgs& a, int seq, int k_head, int v_head)
      : k(static_cast<const __nv_bfloat16*>(a.k_cache) + static_cast<int64_t>(k_head) * a.dim),
        v(static_cast<const __nv_bfloat16*>(a.v_cache) + static_cast<int64_t>(v_head) * a.vdim),
        bt(a.block_table + static_cast<int64_t>(seq) * a.max_blocks), k_pitch(a.k_pitch), v_pitch(a.v_pitch),
        block_size(a.block_size), shift(log2_of(a.block_size)), dim(a.dim), vdim(a.vdim) {}
  __device__ __forceinline__ int64_t slot(int j) const {
    return page_slot(bt, block_size, shift, j);
  }
};
__device__ __forceinline__ void copy8(__nv_bfloat16* d, const __nv_bfloat16* s, int c, int cols) {   // columns c .. c + 7 of a row
  if ((cols & 7) == 0) {
    cp_async16(d, s + c);
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) d[e] = c + e < cols ? s[c + e] : __float2bfloat16_rn(0.0f);
  }
}

}  // namespace nx
