// Causal attention over a paged cache for any head sizes: sliding window, chunks, kept first keys, a sink in the denominator, score
// soft-capping, biases by distance, grouped query heads, different key and value widths (see nx_api_mixers.h).  The query heads that
// share a KV head are packed into the rows of one tensor-core tile, so a KV page is read once for all of them: 128 (token, head) rows
// per block in prompts, up to 16 heads of one token in decoding.  Scores, soft-capping and softmax are FP32; only the products take BF16 operands.
#include "mixer_common.cuh"
#include "nx_api_mixers.h"
#include "paged_keys.cuh"

#include <algorithm>

namespace {
using namespace nx;

constexpr int kKeys = 64;              // keys per shared-memory stage
constexpr int kRows = 128;             // (token, head) rows per block in prompts

// One stage of keys and values into shared memory, each [kKeys][DP + 8]; keys past index `last` and columns past the head size
// become zeros.
template <int DP>
__device__ __forceinline__ void stage_kv(__nv_bfloat16* dst, const KvSource& src, const KeyRange& keys, int k0, int last) {
  constexpr int CH = DP / 8, LD = DP + 8;
  for (int i = threadIdx.x; i < kKeys * CH; i += blockDim.x) {
    const int key = i / CH, c = (i % CH) * 8, j = k0 + key;
    __nv_bfloat16 *dk = dst + key * LD + c, *dv = dk + kKeys * LD;
    const bool in = j <= last;
    const int64_t slot = in ? src.slot(keys.position(j)) : 0;
    if (in && c < src.dim) copy8(dk, src.k + slot * src.k_pitch, c, src.dim);
    else *reinterpret_cast<uint4*>(dk) = make_uint4(0u, 0u, 0u, 0u);
    if (in && c < src.vdim) copy8(dv, src.v + slot * src.v_pitch, c, src.vdim);
    else *reinterpret_cast<uint4*>(dv) = make_uint4(0u, 0u, 0u, 0u);
  }
}

// ------------------------------------------------------------------------------------------------
// prompts: grid (tiles, kv_heads * head tiles, value heads), 8 warps of 16 rows
// ------------------------------------------------------------------------------------------------
template <int DP, bool kBias>
__global__ void __launch_bounds__(kRows * 2)
paged_prefill_kernel(const NxPagedWindowArgs a, int rt, int tq, int head_tiles) {
  constexpr int LD = DP + 8;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* sQ = sm;                       // [kRows][LD]
  __nv_bfloat16* sKV = sQ + kRows * LD;         // [2 stages][K, V][64][LD]
  __shared__ int s_tile[3];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0) {
    int seg = 0, off = 0;
    const bool ok = find_tile(a.seg, tq, blockIdx.x, seg, off);
    if (lane == 0) {
      s_tile[0] = ok;
      s_tile[1] = seg;
      s_tile[2] = off;
    }
  }
  __syncthreads();
  if (!s_tile[0]) return;
  const int sg = s_tile[1], t0 = s_tile[2] * tq;
  const int hk = blockIdx.y / head_tiles, ht = blockIdx.y % head_tiles;
  const int rep = a.heads / a.kv_heads, h0 = hk * rep + ht * rt, nh = min(rt, rep - ht * rt);
  const int nt = min(tq, a.seg.len[sg] - t0);
  const int pos0 = a.seg.pos[sg] + t0;
  const int64_t row0 = static_cast<int64_t>(a.seg.row0[sg]) + t0;
  const KeyRange keys(a, pos0, pos0 + nt - 1);
  const int last = keys.count - 1;
  const KvSource src(a, a.seg.seq[sg], hk, a.all_values ? blockIdx.z : hk);
  auto stage = [&](int k0, int s) {
    stage_kv<DP>(sKV + (s * 2) * kKeys * LD, src, keys, k0, last);
    cp_async_commit();
  };
  stage(0, 0);
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q);
    const float sign = a.scale < 0.0f ? -1.0f : 1.0f;      // the score map wants a positive factor
    const uint32_t flip = a.scale < 0.0f ? 0x80008000u : 0u;
    const bool pairs = ((a.dim | static_cast<int>(a.ldq)) & 1) == 0 && (reinterpret_cast<uintptr_t>(a.q) & 3) == 0;
    for (int i = threadIdx.x; i < kRows * DP / 2; i += kRows * 2) {
      const int m = i / (DP / 2), d = (i % (DP / 2)) * 2, tok = m / rt, hh = m % rt;
      const bool in = tok < nt && hh < nh;
      const __nv_bfloat16* qp = q + (row0 + tok) * a.ldq + static_cast<int64_t>(h0 + hh) * a.dim + d;
      if (pairs) {
        *reinterpret_cast<uint32_t*>(sQ + m * LD + d) = in && d < a.dim ? *reinterpret_cast<const uint32_t*>(qp) ^ flip : 0u;
      } else {
        sQ[m * LD + d] = in && d < a.dim ? __float2bfloat16_rn(sign * __bfloat162float(qp[0])) : __float2bfloat16_rn(0.0f);
        sQ[m * LD + d + 1] = in && d + 1 < a.dim ? __float2bfloat16_rn(sign * __bfloat162float(qp[1])) : __float2bfloat16_rn(0.0f);
      }
    }
  }
  int qpos[2], qlo[2];                          // position of this thread's two rows, -1: padding row; its first key
  const float* brow[2];                         // its head's biases
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int m = warp * 16 + i * 8 + (lane >> 2);
    const bool in = m / rt < nt && m % rt < nh;
    qpos[i] = in ? pos0 + m / rt : -1;
    qlo[i] = in ? first_key(a, qpos[i]) : 0;
    brow[i] = kBias ? a.bias + static_cast<int64_t>(h0 + (in ? m % rt : 0)) * a.bias_len : nullptr;
  }
  // lowest position among the warp's 16 rows; -1 with a padding row among them
  const int warp_lo = __reduce_min_sync(0xffffffffu, min(qpos[0], qpos[1]));
  const int warp_qlo = __reduce_max_sync(0xffffffffu, max(qlo[0], qlo[1]));     // the last first key of a row
  const ScoreMap map(fabsf(a.scale), a.softcap);
  float o[DP / 8][4], mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
#pragma unroll
  for (int i = 0; i < DP / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
  int s = 0;
  for (int k0 = 0; k0 <= last; k0 += kKeys, s ^= 1) {
    if (k0 + kKeys <= last) {
      stage(k0 + kKeys, s ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const __nv_bfloat16* sK = sKV + (s * 2) * kKeys * LD;
    const __nv_bfloat16* sV = sK + kKeys * LD;
    float sc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) sc[n][e] = 0.0f;
#pragma unroll
    for (int kk = 0; kk < DP / 16; ++kk) {
      uint32_t qa[4];
      ldmatrix_x4(qa, smem_addr(sQ + (warp * 16 + (lane & 15)) * LD + kk * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        uint32_t kb[4];
        ldmatrix_x4(kb, smem_addr(sK + (n * 16 + (lane & 7) + ((lane >> 4) << 3)) * LD + kk * 16 + ((lane >> 3) & 1) * 8));
        mma_bf16(sc[2 * n], qa, kb[0], kb[1]);
        mma_bf16(sc[2 * n + 1], qa, kb[2], kb[3]);
      }
    }
    // every row of this warp sees the whole stage, unless it reaches past a row's own position or before its window
    const int p0 = keys.position(k0);
    const bool edge = warp_lo < 0 || keys.position(k0 + kKeys - 1) > warp_lo || p0 < warp_qlo;
    float tmax[2] = {-INFINITY, -INFINITY};
    if constexpr (kBias) {
      const bool far = warp_lo >= 0 && warp_lo - keys.position(k0 + kKeys - 1) >= a.bias_len - 1;
      float b[2] = {0.0f, 0.0f};
      if (far) {
        b[0] = __ldg(brow[0] + a.bias_len - 1);
        b[1] = __ldg(brow[1] + a.bias_len - 1);
      }
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float bias = b[e >> 1];
          if (!far) {
            const int dist = qpos[e >> 1] - keys.position(k0 + n * 8 + (lane & 3) * 2 + (e & 1));
            bias = __ldg(brow[e >> 1] + min(max(dist, 0), a.bias_len - 1));
          }
          sc[n][e] = fmaf(bias, kLog2e, map(sc[n][e]));
        }
    }
    if (edge) {
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = keys.position(k0 + n * 8 + (lane & 3) * 2 + (e & 1));
          if (!(j <= qpos[e >> 1] && (j >= qlo[e >> 1] || j < a.keep_first))) sc[n][e] = -INFINITY;
        }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) tmax[e >> 1] = fmaxf(tmax[e >> 1], sc[n][e]);
    float base[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 1));
      tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 2));
      const float nm = fmaxf(mx[i], kBias ? tmax[i] : map(tmax[i]));
      base[i] = nm == -INFINITY ? 0.0f : nm;
      const float alpha = ex2_approx(mx[i] - base[i]);     // first stage: 2^-inf = 0
      mx[i] = nm;
      sum[i] *= alpha;
#pragma unroll
      for (int n = 0; n < DP / 8; ++n) {
        o[n][2 * i] *= alpha;
        o[n][2 * i + 1] *= alpha;
      }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        sc[n][e] = edge && sc[n][e] == -INFINITY ? 0.0f
                   : kBias                       ? ex2_approx(sc[n][e] - base[e >> 1])
                                                 : map.prob(sc[n][e], base[e >> 1]);
        sum[e >> 1] += sc[n][e];
      }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      const uint32_t pa[4] = {bf16_pair(sc[2 * kk][0], sc[2 * kk][1]), bf16_pair(sc[2 * kk][2], sc[2 * kk][3]),
                              bf16_pair(sc[2 * kk + 1][0], sc[2 * kk + 1][1]), bf16_pair(sc[2 * kk + 1][2], sc[2 * kk + 1][3])};
#pragma unroll
      for (int n = 0; n < DP / 16; ++n) {
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, smem_addr(sV + (kk * 16 + (lane & 15)) * LD + n * 16 + (lane >> 4) * 8));
        mma_bf16(o[2 * n], pa, vb[0], vb[1]);
        mma_bf16(o[2 * n + 1], pa, vb[2], vb[3]);
      }
    }
    __syncthreads();
  }
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out);
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
    sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
    if (qpos[i] < 0) continue;
    const int m = warp * 16 + i * 8 + (lane >> 2);
    const float g = a.gate != nullptr ? a.gate[(row0 + m / rt) * a.heads + h0 + m % rt] : 1.0f;
    if (a.sink != nullptr) sum[i] += exp2f(a.sink[h0 + m % rt] * kLog2e - mx[i]);
    const float inv = a.out_scale * g / sum[i];
    const int64_t slice = a.all_values ? static_cast<int64_t>(h0 + m % rt) * a.kv_heads + blockIdx.z : h0 + m % rt;
    __nv_bfloat16* op = out + (row0 + m / rt) * a.ldo + slice * a.vdim;
#pragma unroll
    for (int n = 0; n < DP / 8; ++n) {
      const int d = n * 8 + (lane & 3) * 2;
      if (d < a.vdim) op[d] = __float2bfloat16_rn(o[n][2 * i] * inv);
      if (d + 1 < a.vdim) op[d + 1] = __float2bfloat16_rn(o[n][2 * i + 1] * inv);
    }
  }
}

// ------------------------------------------------------------------------------------------------
// decoding: grid (segments, kv_heads * head tiles, splits); the 4 warps take 16 keys each of every
// 64-key stage, with their own running softmax, and merge at the end
// ------------------------------------------------------------------------------------------------
template <int DP, bool kBias>
__global__ void __launch_bounds__(128)
paged_decode_mma_kernel(const NxPagedWindowArgs a, int head_tiles) {
  constexpr int LD = DP + 8;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* sQ = sm;                       // [16][LD]
  __nv_bfloat16* sKV = sQ + 16 * LD;            // [2 stages][K, V][64][LD]; the warps' partial outputs afterwards
  __shared__ float s_m[4][16], s_l[4][16];
  const int sg = blockIdx.x;
  if (a.seg.len[sg] <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hk = blockIdx.y / head_tiles, ht = blockIdx.y % head_tiles;
  const int rep = a.heads / a.kv_heads, h0 = hk * rep + ht * 16, nh = min(16, rep - ht * 16);
  const int pos = a.seg.pos[sg];
  const int64_t row = a.seg.row0[sg];
  const KvSource src(a, a.seg.seq[sg], hk, hk);
  const KeyRange keys(a, pos, pos);
  const int per = ((keys.count + kKeys - 1) / kKeys + a.splits - 1) / a.splits * kKeys;
  const int first = static_cast<int>(blockIdx.z) * per, last = min(keys.count, first + per) - 1;
  auto stage = [&](int k0, int s) {
    stage_kv<DP>(sKV + (s * 2) * kKeys * LD, src, keys, k0, last);
    cp_async_commit();
  };
  if (first <= last) stage(first, 0);
  const float sign = a.scale < 0.0f ? -1.0f : 1.0f;
  for (int i = threadIdx.x; i < 16 * DP; i += 128) {
    const int m = i / DP, d = i % DP;
    sQ[m * LD + d] = (m < nh && d < a.dim)
                         ? __float2bfloat16_rn(sign * __bfloat162float(static_cast<const __nv_bfloat16*>(
                               a.q)[row * a.ldq + static_cast<int64_t>(h0 + m) * a.dim + d]))
                         : __float2bfloat16_rn(0.0f);
  }
  const ScoreMap map(fabsf(a.scale), a.softcap);
  float o[DP / 8][4], mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
#pragma unroll
  for (int i = 0; i < DP / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
  int s = 0;
  for (int k0 = first; k0 <= last; k0 += kKeys, s ^= 1) {
    if (k0 + kKeys <= last) {
      stage(k0 + kKeys, s ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    if (k0 + warp * 16 <= last) {
      const __nv_bfloat16* sK = sKV + ((s * 2) * kKeys + warp * 16) * LD;
      const __nv_bfloat16* sV = sK + kKeys * LD;
      float sc[2][4] = {{0.0f, 0.0f, 0.0f, 0.0f}, {0.0f, 0.0f, 0.0f, 0.0f}};
#pragma unroll
      for (int kk = 0; kk < DP / 16; ++kk) {
        uint32_t qa[4], kb[4];
        ldmatrix_x4(qa, smem_addr(sQ + (lane & 15) * LD + kk * 16 + (lane >> 4) * 8));
        ldmatrix_x4(kb, smem_addr(sK + ((lane & 7) + ((lane >> 4) << 3)) * LD + kk * 16 + ((lane >> 3) & 1) * 8));
        mma_bf16(sc[0], qa, kb[0], kb[1]);
        mma_bf16(sc[1], qa, kb[2], kb[3]);
      }
      float tmax[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = k0 + warp * 16 + n * 8 + (lane & 3) * 2 + (e & 1);
          if constexpr (kBias) {
            const int m = min((e >> 1) * 8 + (lane >> 2), nh - 1);
            const int dist = min(max(pos - keys.position(j), 0), a.bias_len - 1);
            sc[n][e] = fmaf(__ldg(a.bias + static_cast<int64_t>(h0 + m) * a.bias_len + dist), kLog2e, map(sc[n][e]));
          }
          sc[n][e] = j <= last ? sc[n][e] : -INFINITY;
          tmax[e >> 1] = fmaxf(tmax[e >> 1], sc[n][e]);
        }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 1));
        tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 2));
        const float nm = fmaxf(mx[i], kBias ? tmax[i] : map(tmax[i]));  // at least one key of this warp is in range
        const float alpha = ex2_approx(mx[i] - nm);
        mx[i] = nm;
        sum[i] *= alpha;
#pragma unroll
        for (int n = 0; n < DP / 8; ++n) {
          o[n][2 * i] *= alpha;
          o[n][2 * i + 1] *= alpha;
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          sc[n][e] = sc[n][e] == -INFINITY ? 0.0f : kBias ? ex2_approx(sc[n][e] - mx[e >> 1]) : map.prob(sc[n][e], mx[e >> 1]);
          sum[e >> 1] += sc[n][e];
        }
      const uint32_t pa[4] = {bf16_pair(sc[0][0], sc[0][1]), bf16_pair(sc[0][2], sc[0][3]), bf16_pair(sc[1][0], sc[1][1]),
                              bf16_pair(sc[1][2], sc[1][3])};
#pragma unroll
      for (int n = 0; n < DP / 16; ++n) {
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, smem_addr(sV + (lane & 15) * LD + n * 16 + (lane >> 4) * 8));
        mma_bf16(o[2 * n], pa, vb[0], vb[1]);
        mma_bf16(o[2 * n + 1], pa, vb[2], vb[3]);
      }
    }
    __syncthreads();
  }
  float* sO = reinterpret_cast<float*>(sKV);    // [4 warps][16][DP]
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
    sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
    const int m = i * 8 + (lane >> 2);
    if ((lane & 3) == 0) {
      s_m[warp][m] = mx[i];
      s_l[warp][m] = sum[i];
    }
#pragma unroll
    for (int n = 0; n < DP / 8; ++n) {
      sO[(warp * 16 + m) * DP + n * 8 + (lane & 3) * 2] = o[n][2 * i];
      sO[(warp * 16 + m) * DP + n * 8 + (lane & 3) * 2 + 1] = o[n][2 * i + 1];
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * a.vdim; i += 128) {
    const int m = i / a.vdim, d = i % a.vdim;
    float gm = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) gm = fmaxf(gm, s_m[w][m]);
    float gl = 0.0f, go = 0.0f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = s_m[w][m] == -INFINITY ? 0.0f : exp2f(s_m[w][m] - gm);
      gl += s_l[w][m] * f;
      go += sO[(w * 16 + m) * DP + d] * f;
    }
    if (a.splits == 1) {
      if (a.sink != nullptr) gl += exp2f(a.sink[h0 + m] * kLog2e - gm);
      const float g = a.gate != nullptr ? a.gate[row * a.heads + h0 + m] : 1.0f;
      static_cast<__nv_bfloat16*>(a.out)[row * a.ldo + static_cast<int64_t>(h0 + m) * a.vdim + d] =
          __float2bfloat16_rn(go / gl * a.out_scale * g);
    } else {
      const int64_t pi = (static_cast<int64_t>(sg) * a.heads + h0 + m) * a.splits + blockIdx.z;
      a.part_o[pi * a.vdim + d] = go;
      if (d == 0) {
        a.part_ml[pi * 2] = gm;
        a.part_ml[pi * 2 + 1] = gl;
      }
    }
  }
}

__global__ void paged_decode_merge_kernel(const NxPagedWindowArgs a) {
  const int sg = blockIdx.x, h = blockIdx.y;
  if (a.seg.len[sg] <= 0) return;
  const int64_t base = (static_cast<int64_t>(sg) * a.heads + h) * a.splits, row = a.seg.row0[sg];
  const float g = a.gate != nullptr ? a.gate[row * a.heads + h] : 1.0f;
  float gm = -INFINITY;
  for (int s = 0; s < a.splits; ++s) gm = fmaxf(gm, a.part_ml[(base + s) * 2]);
  for (int d = threadIdx.x; d < a.vdim; d += blockDim.x) {
    float gl = 0.0f, go = 0.0f;
    for (int s = 0; s < a.splits; ++s) {
      const float m = a.part_ml[(base + s) * 2];
      const float w = m == -INFINITY ? 0.0f : exp2f(m - gm);
      gl += a.part_ml[(base + s) * 2 + 1] * w;
      go += a.part_o[(base + s) * a.vdim + d] * w;
    }
    if (a.sink != nullptr) gl += exp2f(a.sink[h] * kLog2e - gm);
    static_cast<__nv_bfloat16*>(a.out)[row * a.ldo + static_cast<int64_t>(h) * a.vdim + d] =
        __float2bfloat16_rn(go / gl * a.out_scale * g);
  }
}

// ------------------------------------------------------------------------------------------------
// FP32: one block per (row, head), a key per thread for the scores, a value column per thread for the sum
// ------------------------------------------------------------------------------------------------
constexpr int kF32Cols = 8;   // value columns per thread: vdim <= 1024

__global__ void __launch_bounds__(128) paged_window_f32_kernel(const NxPagedWindowArgs a) {
  extern __shared__ __align__(16) float sf[];
  __shared__ float s_red[32];
  __shared__ int64_t s_slot[128];
  float* sQ = sf;               // [dim]
  float* sP = sf + a.dim;       // [128]
  const int nv = a.all_values ? a.kv_heads : 1;
  const int t = blockIdx.x, h = blockIdx.y / nv, sg = blockIdx.z;
  if (t >= a.seg.len[sg]) return;
  const int hk = h / (a.heads / a.kv_heads), pos = a.seg.pos[sg] + t, tid = threadIdx.x;
  const int64_t row = static_cast<int64_t>(a.seg.row0[sg]) + t;
  const int32_t* bt = a.block_table + static_cast<int64_t>(a.seg.seq[sg]) * a.max_blocks;
  const float* kc = static_cast<const float*>(a.k_cache);
  const float* vc = static_cast<const float*>(a.v_cache) + (a.all_values ? blockIdx.y % nv : hk) * a.vdim;
  for (int d = tid; d < a.dim; d += 128) sQ[d] = static_cast<const float*>(a.q)[row * a.ldq + static_cast<int64_t>(h) * a.dim + d];
  float acc[kF32Cols], mx = -INFINITY, sum = 0.0f;
#pragma unroll
  for (int c = 0; c < kF32Cols; ++c) acc[c] = 0.0f;
  const KeyRange keys(a, pos, pos);
  for (int k0 = 0; k0 < keys.count; k0 += 128) {
    __syncthreads();
    float sc = -INFINITY;
    if (k0 + tid < keys.count) {
      const int j = keys.position(k0 + tid);
      const int64_t slot = static_cast<int64_t>(bt[j / a.block_size]) * a.block_size + j % a.block_size;
      s_slot[tid] = slot;
      const float* k = kc + slot * a.k_pitch + hk * a.dim;
      float s = 0.0f;
      for (int d = 0; d < a.dim; ++d) s += sQ[d] * k[d];
      sc = s * a.scale;
      if (a.softcap > 0.0f) sc = a.softcap * tanhf(sc / a.softcap);
      if (a.bias != nullptr) sc += a.bias[static_cast<int64_t>(h) * a.bias_len + min(pos - j, a.bias_len - 1)];
    }
    const float nm = fmaxf(mx, block_max(sc, s_red));
    const float p = expf(sc - nm), alpha = expf(mx - nm);
    mx = nm;
    sP[tid] = p;
    sum = sum * alpha + block_sum(p, s_red);     // the barriers inside publish sP and s_slot
    const int n = min(128, keys.count - k0);
#pragma unroll
    for (int c = 0; c < kF32Cols; ++c) {
      const int d = tid + c * 128;
      if (d < a.vdim) {
        float v = acc[c] * alpha;
        for (int i = 0; i < n; ++i) v += sP[i] * vc[s_slot[i] * a.v_pitch + d];
        acc[c] = v;
      }
    }
  }
  const float g = a.gate != nullptr ? a.gate[row * a.heads + h] : 1.0f;
  if (a.sink != nullptr) sum += expf(a.sink[h] - mx);
  for (int c = 0; c < kF32Cols; ++c) {
    const int d = tid + c * 128;
    if (d < a.vdim) static_cast<float*>(a.out)[row * a.ldo + static_cast<int64_t>(blockIdx.y) * a.vdim + d] = acc[c] / sum * (a.out_scale * g);
  }
}

int check_paged(const NxPagedWindowArgs* a, int dtype) {
  if (a == nullptr || a->dtype != dtype || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads) return -1;
  if (a->keep_first < 0 || a->dim <= 0 || a->vdim <= 0 || a->block_size <= 0 || a->max_blocks <= 0 || a->seg.count > 65535) return -1;
  if (a->chunk < 0 || (a->bias != nullptr && a->bias_len <= 0)) return -1;
  if (a->k_pitch < static_cast<int64_t>(a->kv_heads) * a->dim || a->v_pitch < static_cast<int64_t>(a->kv_heads) * a->vdim) return -1;
  return 0;
}
int padded_dim(const NxPagedWindowArgs* a) {
  const int d = std::max(a->dim, a->vdim);
  return d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : d <= 256 ? 256 : 0;
}

template <int DP, bool kBias>
int launch_prefill_as(const NxPagedWindowArgs* a, dim3 grid, int rt, int tq, int head_tiles, cudaStream_t st) {
  constexpr int kSmem = (kRows + 4 * kKeys) * (DP + 8) * 2;
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(paged_prefill_kernel<DP, kBias>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem) != cudaSuccess) return -2;
    once = true;
  }
  paged_prefill_kernel<DP, kBias><<<grid, kRows * 2, kSmem, st>>>(*a, rt, tq, head_tiles);
  return launch_status();
}
template <int DP>
int launch_prefill(const NxPagedWindowArgs* a, dim3 grid, int rt, int tq, int head_tiles, cudaStream_t st) {
  return a->bias != nullptr ? launch_prefill_as<DP, true>(a, grid, rt, tq, head_tiles, st)
                            : launch_prefill_as<DP, false>(a, grid, rt, tq, head_tiles, st);
}

template <int DP, bool kBias>
int launch_decode_as(const NxPagedWindowArgs* a, dim3 grid, int head_tiles, cudaStream_t st) {
  constexpr int kSmem = (16 + 4 * kKeys) * (DP + 8) * 2;
  static_assert(4 * kKeys * (DP + 8) * 2 >= 4 * 16 * DP * 4, "partial outputs reuse the stages");
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(paged_decode_mma_kernel<DP, kBias>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem) != cudaSuccess) return -2;
    once = true;
  }
  paged_decode_mma_kernel<DP, kBias><<<grid, 128, kSmem, st>>>(*a, head_tiles);
  return launch_status();
}
template <int DP>
int launch_decode(const NxPagedWindowArgs* a, dim3 grid, int head_tiles, cudaStream_t st) {
  return a->bias != nullptr ? launch_decode_as<DP, true>(a, grid, head_tiles, st) : launch_decode_as<DP, false>(a, grid, head_tiles, st);
}

}  // namespace

extern "C" int nx_paged_window_prefill(const NxPagedWindowArgs* a, nx_stream_t stream) {
  if (check_paged(a, NX_BF16)) return -1;
  if (a->seg.count <= 0 || a->seg.total_len <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int rep = a->heads / a->kv_heads;
  const int rt = std::min(rep, 16), head_tiles = (rep + rt - 1) / rt, tq = kRows / rt;
  dim3 grid(a->seg.total_len / tq + a->seg.count, a->kv_heads * head_tiles, a->all_values ? a->kv_heads : 1);
  switch (padded_dim(a)) {
    case 32: return launch_prefill<32>(a, grid, rt, tq, head_tiles, st);
    case 64: return launch_prefill<64>(a, grid, rt, tq, head_tiles, st);
    case 128: return launch_prefill<128>(a, grid, rt, tq, head_tiles, st);
    case 256: return launch_prefill<256>(a, grid, rt, tq, head_tiles, st);
    default: return -1;
  }
}

extern "C" int nx_paged_window_decode(const NxPagedWindowArgs* a, nx_stream_t stream) {
  if (check_paged(a, NX_BF16) || a->splits < 1 || a->splits > 65535 || a->all_values) return -1;
  if (a->splits > 1 && (a->part_o == nullptr || a->part_ml == nullptr)) return -1;
  if (a->seg.count <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int rep = a->heads / a->kv_heads, head_tiles = (rep + 15) / 16;
  dim3 grid(a->seg.count, a->kv_heads * head_tiles, a->splits);
  int rc = -1;
  switch (padded_dim(a)) {
    case 32: rc = launch_decode<32>(a, grid, head_tiles, st); break;
    case 64: rc = launch_decode<64>(a, grid, head_tiles, st); break;
    case 128: rc = launch_decode<128>(a, grid, head_tiles, st); break;
    case 256: rc = launch_decode<256>(a, grid, head_tiles, st); break;
    default: return -1;
  }
  if (rc == 0 && a->splits > 1) {
    paged_decode_merge_kernel<<<dim3(a->seg.count, a->heads), std::min(256, (a->vdim + 31) / 32 * 32), 0, st>>>(*a);
    rc = launch_status();
  }
  return rc;
}

extern "C" int nx_paged_window_f32(const NxPagedWindowArgs* a, nx_stream_t stream) {
  if (check_paged(a, NX_F32) || a->vdim > 128 * kF32Cols || a->dim > 4096) return -1;
  if (a->seg.count <= 0 || a->seg.max_len <= 0) return 0;
  dim3 grid(a->seg.max_len, a->heads * (a->all_values ? a->kv_heads : 1), a->seg.count);
  paged_window_f32_kernel<<<grid, 128, (a->dim + 128) * sizeof(float), static_cast<cudaStream_t>(stream)>>>(*a);
  return launch_status();
}
