// Decoding with heads that mix their weights after the softmax (see nx_api_mixers.h).  A row's weight for a key is a mixture over all
// heads, so the values of a KV head need the scores of every query head.  Two kernels: scores of all heads (FP32, every key read
// once) with the running maximum and sum of each span of keys; then, per KV head, the normalised weights of all heads for 64 keys at
// a time, their mixture for the heads of this KV head (FP32) and the product with the values.  A key's scores are a few per cent of
// the bytes of its keys and values.
#include "mixer_common.cuh"
#include "nx_api_mixers.h"
#include "paged_keys.cuh"

#include <algorithm>

namespace {
using namespace nx;

constexpr int kKeys = 64;              // keys per shared-memory stage

// the span of keys that block z of `splits` takes: first .. last (empty: first > last)
__device__ __forceinline__ void key_span(const NxPagedWindowArgs& a, const KeyRange& keys, int z, int& first, int& last) {
  const int per = ((keys.count + kKeys - 1) / kKeys + a.splits - 1) / a.splits * kKeys;
  first = z * per;
  last = min(keys.count, first + per) - 1;
}

// keys (or values) first .. of one stage into shared memory [kKeys][LD]; keys past `last` and columns past `cols` become zeros
template <int DP>
__device__ __forceinline__ void stage_rows(__nv_bfloat16* dst, const __nv_bfloat16* src, int64_t pitch, int cols, const KvSource& at,
                                           const KeyRange& keys, int k0, int last) {
  constexpr int CH = DP / 8, LD = DP + 8;
  for (int i = threadIdx.x; i < kKeys * CH; i += blockDim.x) {
    const int key = i / CH, c = (i % CH) * 8, j = k0 + key;
    __nv_bfloat16* d = dst + key * LD + c;
    if (j <= last && c < cols) copy8(d, src + at.slot(keys.position(j)) * pitch, c, cols);
    else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
  }
}

// ------------------------------------------------------------------------------------------------
// scores: grid (segments, kv_heads * head tiles, splits); a warp takes 16 keys of every stage
// ------------------------------------------------------------------------------------------------
template <int DP>
__global__ void __launch_bounds__(128)
talk_scores_kernel(const NxTalkDecodeArgs t, int head_tiles) {
  constexpr int LD = DP + 8;
  const NxPagedWindowArgs& a = t.base;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* sQ = sm;                       // [16][LD]
  __nv_bfloat16* sK = sQ + 16 * LD;             // [2 stages][64][LD]
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
  int first, last;
  key_span(a, keys, blockIdx.z, first, last);
  auto stage = [&](int k0, int s) {
    stage_rows<DP>(sK + s * kKeys * LD, src.k, src.k_pitch, a.dim, src, keys, k0, last);
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
  float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
  const int m0 = lane >> 2;
  const float* brow[2];
  float* srow[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int m = min(m0 + i * 8, nh - 1);
    brow[i] = a.bias != nullptr ? a.bias + static_cast<int64_t>(h0 + m) * a.bias_len : nullptr;
    srow[i] = t.scores + (static_cast<int64_t>(sg) * a.heads + h0 + m) * t.score_pitch;
  }
  int s = 0;
  for (int k0 = first; k0 <= last; k0 += kKeys, s ^= 1) {
    if (k0 + kKeys <= last) {
      stage(k0 + kKeys, s ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const int kw = k0 + warp * 16;
    if (kw <= last) {
      const __nv_bfloat16* sk = sK + (s * kKeys + warp * 16) * LD;
      float sc[2][4] = {{0.0f, 0.0f, 0.0f, 0.0f}, {0.0f, 0.0f, 0.0f, 0.0f}};
#pragma unroll
      for (int kk = 0; kk < DP / 16; ++kk) {
        uint32_t qa[4], kb[4];
        ldmatrix_x4(qa, smem_addr(sQ + (lane & 15) * LD + kk * 16 + (lane >> 4) * 8));
        ldmatrix_x4(kb, smem_addr(sk + ((lane & 7) + ((lane >> 4) << 3)) * LD + kk * 16 + ((lane >> 3) & 1) * 8));
        mma_bf16(sc[0], qa, kb[0], kb[1]);
        mma_bf16(sc[1], qa, kb[2], kb[3]);
      }
      float tmax[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = kw + n * 8 + (lane & 3) * 2 + (e & 1);
          float v = map(sc[n][e]);
          if (a.bias != nullptr) v = fmaf(__ldg(brow[e >> 1] + min(max(pos - keys.position(j), 0), a.bias_len - 1)), kLog2e, v);
          sc[n][e] = j <= last ? v : -INFINITY;
          tmax[e >> 1] = fmaxf(tmax[e >> 1], sc[n][e]);
        }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        if (m0 + i * 8 < nh) {
#pragma unroll
          for (int n = 0; n < 2; ++n)
            *reinterpret_cast<float2*>(srow[i] + kw + n * 8 + (lane & 3) * 2) = make_float2(sc[n][2 * i], sc[n][2 * i + 1]);
        }
        tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 1));
        tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 2));
        const float nm = fmaxf(mx[i], tmax[i]);       // at least one key of this warp is in range
        sum[i] *= ex2_approx(mx[i] - nm);
        mx[i] = nm;
#pragma unroll
        for (int n = 0; n < 2; ++n) sum[i] += ex2_approx(sc[n][2 * i] - nm) + ex2_approx(sc[n][2 * i + 1] - nm);
      }
    } else {                                           // a whole stage is read later: nothing of it stays undefined
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        if (m0 + i * 8 >= nh) continue;
#pragma unroll
        for (int n = 0; n < 2; ++n)
          *reinterpret_cast<float2*>(srow[i] + kw + n * 8 + (lane & 3) * 2) = make_float2(-INFINITY, -INFINITY);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
    sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
    if ((lane & 3) == 0) {
      s_m[warp][m0 + i * 8] = mx[i];
      s_l[warp][m0 + i * 8] = sum[i];
    }
  }
  __syncthreads();
  if (threadIdx.x < nh) {
    const int m = threadIdx.x;
    float gm = -INFINITY, gl = 0.0f;
#pragma unroll
    for (int w = 0; w < 4; ++w) gm = fmaxf(gm, s_m[w][m]);
#pragma unroll
    for (int w = 0; w < 4; ++w) gl += s_m[w][m] == -INFINITY ? 0.0f : s_l[w][m] * exp2f(s_m[w][m] - gm);
    float* ml = a.part_ml + ((static_cast<int64_t>(sg) * a.heads + h0 + m) * a.splits + blockIdx.z) * 2;
    ml[0] = gm;
    ml[1] = gl;
  }
}

// ------------------------------------------------------------------------------------------------
// mixture and values: grid (segments, kv_heads * head tiles, splits); a warp takes DP / 4 value columns
// ------------------------------------------------------------------------------------------------
template <int DP>
__global__ void __launch_bounds__(128)
talk_values_kernel(const NxTalkDecodeArgs t, int head_tiles) {
  constexpr int LD = DP + 8, LW = kKeys + 8, COLS = DP / 4;
  const NxPagedWindowArgs& a = t.base;
  const int H = a.heads;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* sV = sm;                                            // [2 stages][64][LD]
  __nv_bfloat16* sW = sV + 2 * kKeys * LD;                           // [16][LW] mixed weights
  float* sS = reinterpret_cast<float*>(sW + 16 * LW);                // [2 stages][H][64] scores
  float* sT = sS + 2 * H * kKeys;                                    // [H][16]: talk of this block's heads, from every head
  float* sN = sT + H * 16;                                           // [H]: log2 of the sum over all keys
  const int sg = blockIdx.x;
  if (a.seg.len[sg] <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hk = blockIdx.y / head_tiles, ht = blockIdx.y % head_tiles;
  const int rep = H / a.kv_heads, h0 = hk * rep + ht * 16, nh = min(16, rep - ht * 16);
  const int pos = a.seg.pos[sg];
  const int64_t row = a.seg.row0[sg];
  const KvSource src(a, a.seg.seq[sg], hk, hk);
  const KeyRange keys(a, pos, pos);
  int first, last;
  key_span(a, keys, blockIdx.z, first, last);
  const float* scores = t.scores + static_cast<int64_t>(sg) * H * t.score_pitch;
  auto stage = [&](int k0, int s) {
    stage_rows<DP>(sV + s * kKeys * LD, src.v, src.v_pitch, a.vdim, src, keys, k0, last);
    for (int i = threadIdx.x; i < H * (kKeys / 4); i += 128) {
      const int g = i / (kKeys / 4), c = (i % (kKeys / 4)) * 4;
      cp_async16(sS + (s * H + g) * kKeys + c, scores + g * t.score_pitch + k0 + c);
    }
    cp_async_commit();
  };
  if (first <= last) stage(first, 0);
  for (int i = threadIdx.x; i < H * 16; i += 128) sT[i] = i % 16 < nh ? t.talk[(h0 + i % 16) * H + i / 16] : 0.0f;
  for (int i = threadIdx.x; i < 16 * LW; i += 128) sW[i] = __float2bfloat16_rn(0.0f);
  for (int g = threadIdx.x; g < H; g += 128) {
    const float* ml = a.part_ml + (static_cast<int64_t>(sg) * H + g) * a.splits * 2;
    float gm = -INFINITY, gl = 0.0f;
    for (int z = 0; z < a.splits; ++z) gm = fmaxf(gm, ml[2 * z]);
    for (int z = 0; z < a.splits; ++z) gl += ml[2 * z] == -INFINITY ? 0.0f : ml[2 * z + 1] * exp2f(ml[2 * z] - gm);
    sN[g] = gm + log2f(gl);
  }
  float o[COLS / 8][4];
#pragma unroll
  for (int i = 0; i < COLS / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.0f;
  const int key = threadIdx.x & 63, per = (nh + 1) / 2, m0 = (threadIdx.x >> 6) * per, mn = min(per, nh - m0);   // up to 8 heads of one key
  int s = 0;
  for (int k0 = first; k0 <= last; k0 += kKeys, s ^= 1) {
    if (k0 + kKeys <= last) {
      stage(k0 + kKeys, s ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    {
      float w[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) w[i] = 0.0f;
      const float* sc = sS + s * H * kKeys + key;
#pragma unroll 4
      for (int g = 0; g < H; ++g) {
        const float p = ex2_approx(sc[g * kKeys] - sN[g]);
        const float* tg = sT + g * 16 + m0;
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (i < mn) w[i] = fmaf(tg[i], p, w[i]);
      }
      if (k0 + key > last) {
#pragma unroll
        for (int i = 0; i < 8; ++i) w[i] = 0.0f;
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i < mn) sW[(m0 + i) * LW + key] = __float2bfloat16_rn(w[i]);
    }
    __syncthreads();
    const __nv_bfloat16* sv = sV + s * kKeys * LD + warp * COLS;
#pragma unroll
    for (int kk = 0; kk < kKeys / 16; ++kk) {
      uint32_t wa[4];
      ldmatrix_x4(wa, smem_addr(sW + (lane & 15) * LW + kk * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int n = 0; n < COLS / 16; ++n) {
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, smem_addr(sv + (kk * 16 + (lane & 15)) * LD + n * 16 + (lane >> 4) * 8));
        mma_bf16(o[2 * n], wa, vb[0], vb[1]);
        mma_bf16(o[2 * n + 1], wa, vb[2], vb[3]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int m = i * 8 + (lane >> 2);
    if (m >= nh) continue;
    const int h = h0 + m;
    const float g = a.splits == 1 ? a.out_scale * (a.gate != nullptr ? a.gate[row * H + h] : 1.0f) : 1.0f;
#pragma unroll
    for (int n = 0; n < COLS / 8; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = warp * COLS + n * 8 + (lane & 3) * 2 + e;
        if (d >= a.vdim) continue;
        const float v = o[n][2 * i + e] * g;
        if (a.splits == 1)
          static_cast<__nv_bfloat16*>(a.out)[row * a.ldo + static_cast<int64_t>(h) * a.vdim + d] = __float2bfloat16_rn(v);
        else
          a.part_o[((static_cast<int64_t>(sg) * H + h) * a.splits + blockIdx.z) * a.vdim + d] = v;
      }
  }
}

// the spans' weights are normalised: their products are added up
__global__ void talk_sum_kernel(const NxPagedWindowArgs a) {
  const int sg = blockIdx.x, h = blockIdx.y;
  if (a.seg.len[sg] <= 0) return;
  const int64_t row = a.seg.row0[sg];
  const float g = a.out_scale * (a.gate != nullptr ? a.gate[row * a.heads + h] : 1.0f);
  const float* p = a.part_o + (static_cast<int64_t>(sg) * a.heads + h) * a.splits * a.vdim;
  for (int d = threadIdx.x; d < a.vdim; d += blockDim.x) {
    float v = 0.0f;
    for (int s = 0; s < a.splits; ++s) v += p[static_cast<int64_t>(s) * a.vdim + d];
    static_cast<__nv_bfloat16*>(a.out)[row * a.ldo + static_cast<int64_t>(h) * a.vdim + d] = __float2bfloat16_rn(v * g);
  }
}

template <int DP>
int launch_scores(const NxTalkDecodeArgs* t, dim3 grid, int head_tiles, cudaStream_t st) {
  constexpr int kSmem = (16 + 2 * kKeys) * (DP + 8) * 2;
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(talk_scores_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem) != cudaSuccess) return -2;
    once = true;
  }
  talk_scores_kernel<DP><<<grid, 128, kSmem, st>>>(*t, head_tiles);
  return launch_status();
}
template <int DP>
int launch_values(const NxTalkDecodeArgs* t, dim3 grid, int head_tiles, cudaStream_t st) {
  constexpr int kFixed = 2 * kKeys * (DP + 8) * 2 + 16 * (kKeys + 8) * 2;
  constexpr int kMost = kFixed + 96 * (2 * kKeys + 17) * 4;
  static_assert(kMost <= 227 * 1024, "shared memory");
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(talk_values_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMost) != cudaSuccess) return -2;
    once = true;
  }
  talk_values_kernel<DP><<<grid, 128, kFixed + t->base.heads * (2 * kKeys + 17) * 4, st>>>(*t, head_tiles);
  return launch_status();
}

}  // namespace

extern "C" int nx_talk_decode(const NxTalkDecodeArgs* t, nx_stream_t stream) {
  if (t == nullptr || t->talk == nullptr || t->scores == nullptr || t->score_pitch <= 0 || t->score_pitch % kKeys) return -1;
  const NxPagedWindowArgs* a = &t->base;
  if (a->dtype != NX_BF16 || a->heads <= 0 || a->heads > 96 || a->kv_heads <= 0 || a->heads % a->kv_heads) return -1;
  if (a->dim <= 0 || a->dim > 256 || a->vdim <= 0 || a->vdim > 256 || a->block_size <= 0 || a->max_blocks <= 0) return -1;
  if (a->splits < 1 || a->splits > 65535 || a->part_ml == nullptr || (a->splits > 1 && a->part_o == nullptr)) return -1;
  if (a->sink != nullptr || a->all_values || a->keep_first < 0 || a->chunk < 0 || (a->bias != nullptr && a->bias_len <= 0)) return -1;
  if (a->k_pitch < static_cast<int64_t>(a->kv_heads) * a->dim || a->v_pitch < static_cast<int64_t>(a->kv_heads) * a->vdim) return -1;
  if (reinterpret_cast<uintptr_t>(t->scores) & 15) return -1;
  if (a->seg.count <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int rep = a->heads / a->kv_heads, head_tiles = (rep + 15) / 16;
  const dim3 grid(a->seg.count, a->kv_heads * head_tiles, a->splits);
  int rc = a->dim <= 64 ? launch_scores<64>(t, grid, head_tiles, st) : a->dim <= 128 ? launch_scores<128>(t, grid, head_tiles, st)
                                                                                      : launch_scores<256>(t, grid, head_tiles, st);
  if (rc) return rc;
  rc = a->vdim <= 64 ? launch_values<64>(t, grid, head_tiles, st) : a->vdim <= 128 ? launch_values<128>(t, grid, head_tiles, st)
                                                                                   : launch_values<256>(t, grid, head_tiles, st);
  if (rc == 0 && a->splits > 1) {
    talk_sum_kernel<<<dim3(a->seg.count, a->heads), std::min(256, (a->vdim + 31) / 32 * 32), 0, st>>>(*a);
    rc = launch_status();
  }
  return rc;
}
