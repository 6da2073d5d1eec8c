// Decoding and short segments with heads that mix their weights after the softmax (see nx_api_mixers.h).  A row's weight for a key is a
// mixture over all heads, so the values of a KV head need the scores of every query head.  Three kernels over a scratch of one score
// and one weight per (row, head, key), a few per cent of the bytes of the keys and values:
//   scores   rows of one KV head against its keys, FP32 scores with the maximum and sum of each span of keys
//   mixture  per row and 64 keys: the normalised weights of all heads, mixed (FP32), as the BF16 operand of the products
//   values   rows of one KV head: weights times values; spans of keys are added up by a fourth kernel
// A tile is 16, 32 or 64 (token, head) rows of one KV head; keys and values are read once per tile.
#include "mixer_common.cuh"
#include "nx_api_mixers.h"
#include "paged_keys.cuh"

#include <algorithm>

namespace {
using namespace nx;

constexpr int kKeys = 64;              // keys per shared-memory stage
constexpr int kThreads = 128;

struct Tile {
  int sg, t0, nt;                      // segment, first token, tokens
  bool ok;
};
// tile `index` of `tq` tokens; with one-row segments tile and segment are the same
__device__ __forceinline__ Tile locate(const NxSegments& seg, int tq, int index, int (&shared)[3]) {
  Tile t;
  if (seg.max_len == 1) {
    t.sg = index;
    t.t0 = 0;
    t.ok = seg.len[index] > 0;
    t.nt = 1;
    return t;
  }
  if (threadIdx.x < 32) {
    int s = 0, off = 0;
    const bool ok = find_tile(seg, tq, index, s, off);
    if (threadIdx.x == 0) {
      shared[0] = ok;
      shared[1] = s;
      shared[2] = off * tq;
    }
  }
  __syncthreads();
  t.ok = shared[0];
  t.sg = shared[1];
  t.t0 = shared[2];
  t.nt = t.ok ? min(tq, seg.len[t.sg] - t.t0) : 0;
  return t;
}

// the span of keys that block z of `splits` takes: first .. last (empty: first > last)
__device__ __forceinline__ void key_span(const NxPagedWindowArgs& a, const KeyRange& keys, int z, int& first, int& last) {
  const int per = ((keys.count + kKeys - 1) / kKeys + a.splits - 1) / a.splits * kKeys;
  first = z * per;
  last = min(keys.count, first + per) - 1;
}

// keys (or values) of one stage into shared memory [kKeys][DP + 8]; keys past `last` and columns past `cols` become zeros
template <int DP>
__device__ __forceinline__ void stage_rows(__nv_bfloat16* dst, const __nv_bfloat16* src, int64_t pitch, int cols, const KvSource& at,
                                           const KeyRange& keys, int k0, int last) {
  constexpr int CH = DP / 8, LD = DP + 8;
  for (int i = threadIdx.x; i < kKeys * CH; i += kThreads) {
    const int key = i / CH, c = (i % CH) * 8, j = k0 + key;
    __nv_bfloat16* d = dst + key * LD + c;
    if (j <= last && c < cols) copy8(d, src + at.slot(keys.position(j)) * pitch, c, cols);
    else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
  }
}

// ------------------------------------------------------------------------------------------------
// scores: grid (tiles, kv_heads * head tiles, splits); MT * 16 rows, a warp takes 16 keys of every stage
// ------------------------------------------------------------------------------------------------
template <int DP, int MT>
__global__ void __launch_bounds__(kThreads)
talk_scores_kernel(const NxTalkPagedArgs t, int rt, int tq, int head_tiles) {
  constexpr int LD = DP + 8, R = MT * 16;
  const NxPagedWindowArgs& a = t.base;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* sQ = sm;                       // [R][LD]
  __nv_bfloat16* sK = sQ + R * LD;              // [2 stages][64][LD]
  __shared__ float s_m[4][R], s_l[4][R];
  __shared__ int s_tile[3];
  const Tile tile = locate(a.seg, tq, blockIdx.x, s_tile);
  if (!tile.ok) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hk = blockIdx.y / head_tiles, ht = blockIdx.y % head_tiles;
  const int rep = a.heads / a.kv_heads, h0 = hk * rep + ht * rt, nh = min(rt, rep - ht * rt);
  const int pos0 = a.seg.pos[tile.sg] + tile.t0;
  const int64_t row0 = static_cast<int64_t>(a.seg.row0[tile.sg]) + tile.t0, scratch0 = static_cast<int64_t>(blockIdx.x) * tq;
  const KvSource src(a, a.seg.seq[tile.sg], hk, hk);
  const KeyRange keys(a, pos0, pos0 + tile.nt - 1);
  int first, last;
  key_span(a, keys, blockIdx.z, first, last);
  auto stage = [&](int k0, int s) {
    stage_rows<DP>(sK + s * kKeys * LD, src.k, src.k_pitch, a.dim, src, keys, k0, last);
    cp_async_commit();
  };
  if (first <= last) stage(first, 0);
  const float sign = a.scale < 0.0f ? -1.0f : 1.0f;
  for (int i = threadIdx.x; i < R * DP; i += kThreads) {
    const int m = i / DP, d = i % DP, tok = m / rt, hh = m % rt;
    sQ[m * LD + d] = (tok < tile.nt && hh < nh && d < a.dim)
                         ? __float2bfloat16_rn(sign * __bfloat162float(static_cast<const __nv_bfloat16*>(
                               a.q)[(row0 + tok) * a.ldq + static_cast<int64_t>(h0 + hh) * a.dim + d]))
                         : __float2bfloat16_rn(0.0f);
  }
  const ScoreMap map(fabsf(a.scale), a.softcap);
  float mx[MT][2], sum[MT][2];
  int qpos[MT][2], qlo[MT][2], bias0[MT][2];    // position (-1: padding row), first key, offset of the head's biases
  float* srow[MT][2];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int m = mt * 16 + i * 8 + (lane >> 2), tok = m / rt, hh = m % rt;
      const bool in = tok < tile.nt && hh < nh;
      mx[mt][i] = -INFINITY;
      sum[mt][i] = 0.0f;
      qpos[mt][i] = in ? pos0 + tok : -1;
      qlo[mt][i] = in ? first_key(a, pos0 + tok) : 0;
      bias0[mt][i] = in ? (h0 + hh) * a.bias_len : 0;
      srow[mt][i] = in ? t.scores + ((scratch0 + tok) * a.heads + h0 + hh) * t.pitch : nullptr;
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
    const __nv_bfloat16* sk = sK + (s * kKeys + warp * 16) * LD;
    float sc[MT][2][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[mt][n][e] = 0.0f;
    if (kw <= last) {
#pragma unroll
      for (int kk = 0; kk < DP / 16; ++kk) {
        uint32_t kb[4];
        ldmatrix_x4(kb, smem_addr(sk + ((lane & 7) + ((lane >> 4) << 3)) * LD + kk * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          uint32_t qa[4];
          ldmatrix_x4(qa, smem_addr(sQ + (mt * 16 + (lane & 15)) * LD + kk * 16 + (lane >> 4) * 8));
          mma_bf16(sc[mt][0], qa, kb[0], kb[1]);
          mma_bf16(sc[mt][1], qa, kb[2], kb[3]);
        }
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const int j0 = kw + n * 8 + (lane & 3) * 2;
      const int p[2] = {keys.position(j0), keys.position(j0 + 1)};
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = e >> 1, pk = p[e & 1];
          float v = map(sc[mt][n][e]);
          if (a.bias != nullptr) v = fmaf(__ldg(a.bias + bias0[mt][i] + min(max(qpos[mt][i] - pk, 0), a.bias_len - 1)), kLog2e, v);
          const bool see = j0 + (e & 1) <= last && pk <= qpos[mt][i] && (pk >= qlo[mt][i] || pk < a.keep_first);
          sc[mt][n][e] = see ? v : -INFINITY;
        }
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < 2; ++i)     // the whole stage is written: it is read as a whole
          if (srow[mt][i] != nullptr) *reinterpret_cast<float2*>(srow[mt][i] + j0) = make_float2(sc[mt][n][2 * i], sc[mt][n][2 * i + 1]);
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        float tmax = fmaxf(fmaxf(sc[mt][0][2 * i], sc[mt][0][2 * i + 1]), fmaxf(sc[mt][1][2 * i], sc[mt][1][2 * i + 1]));
        tmax = fmaxf(tmax, __shfl_xor_sync(0xffffffffu, tmax, 1));
        tmax = fmaxf(tmax, __shfl_xor_sync(0xffffffffu, tmax, 2));
        const float nm = fmaxf(mx[mt][i], tmax), base = nm == -INFINITY ? 0.0f : nm;
        sum[mt][i] *= ex2_approx(mx[mt][i] - base);
        mx[mt][i] = nm;
#pragma unroll
        for (int n = 0; n < 2; ++n) sum[mt][i] += ex2_approx(sc[mt][n][2 * i] - base) + ex2_approx(sc[mt][n][2 * i + 1] - base);
      }
    __syncthreads();
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      sum[mt][i] += __shfl_xor_sync(0xffffffffu, sum[mt][i], 1);
      sum[mt][i] += __shfl_xor_sync(0xffffffffu, sum[mt][i], 2);
      if ((lane & 3) == 0) {
        s_m[warp][mt * 16 + i * 8 + (lane >> 2)] = mx[mt][i];
        s_l[warp][mt * 16 + i * 8 + (lane >> 2)] = sum[mt][i];
      }
    }
  __syncthreads();
  for (int m = threadIdx.x; m < R; m += kThreads) {
    const int tok = m / rt, hh = m % rt;
    if (tok >= tile.nt || hh >= nh) continue;
    float gm = -INFINITY, gl = 0.0f;
#pragma unroll
    for (int w = 0; w < 4; ++w) gm = fmaxf(gm, s_m[w][m]);
#pragma unroll
    for (int w = 0; w < 4; ++w) gl += s_m[w][m] == -INFINITY ? 0.0f : s_l[w][m] * exp2f(s_m[w][m] - gm);
    float* ml = a.part_ml + (((scratch0 + tok) * a.heads + h0 + hh) * a.splits + blockIdx.z) * 2;
    ml[0] = gm;
    ml[1] = gl;
  }
}

// ------------------------------------------------------------------------------------------------
// mixture: grid (scratch rows, blocks of 64 keys in strides); a thread forms up to 8 heads of one key
// ------------------------------------------------------------------------------------------------
constexpr int kMixThreads = 256, kMixHeads = 8;

__global__ void __launch_bounds__(kMixThreads)
talk_mix_kernel(const NxTalkPagedArgs t, int tq) {
  const NxPagedWindowArgs& a = t.base;
  const int H = a.heads, HP = (H + 3) & ~3;
  extern __shared__ __align__(16) float sf[];
  float* sT = sf;                      // [H][HP]: talk, from head, to head
  float* sP = sT + H * HP;             // [H][64] weights
  float* sN = sP + H * kKeys;          // [H] log2 of the sum over all keys
  __shared__ int s_tile[3];
  const Tile tile = locate(a.seg, tq, blockIdx.x / tq, s_tile);
  const int tok = blockIdx.x % tq;
  if (!tile.ok || tok >= tile.nt) return;
  const int pos0 = a.seg.pos[tile.sg] + tile.t0;
  const KeyRange keys(a, pos0, pos0 + tile.nt - 1);
  const int64_t row = static_cast<int64_t>(blockIdx.x) * H;
  for (int i = threadIdx.x; i < H * HP; i += kMixThreads) sT[i] = i % HP < H ? t.talk[(i % HP) * H + i / HP] : 0.0f;
  for (int g = threadIdx.x; g < H; g += kMixThreads) {
    const float* ml = a.part_ml + (row + g) * a.splits * 2;
    float gm = -INFINITY, gl = 0.0f;
    for (int z = 0; z < a.splits; ++z) gm = fmaxf(gm, ml[2 * z]);
    for (int z = 0; z < a.splits; ++z) gl += ml[2 * z] == -INFINITY ? 0.0f : ml[2 * z + 1] * exp2f(ml[2 * z] - gm);
    sN[g] = gm + log2f(gl);
  }
  __syncthreads();
  const int key = threadIdx.x & (kKeys - 1), part = threadIdx.x / kKeys;
  constexpr int kParts = kMixThreads / kKeys;
  for (int k0 = blockIdx.y * kKeys; k0 < keys.count; k0 += gridDim.y * kKeys) {
    for (int g = part; g < H; g += kParts) sP[g * kKeys + key] = ex2_approx(t.scores[(row + g) * t.pitch + k0 + key] - sN[g]);
    __syncthreads();
    for (int h0 = part * kMixHeads; h0 < H; h0 += kParts * kMixHeads) {
      float w[kMixHeads];
#pragma unroll
      for (int i = 0; i < kMixHeads; ++i) w[i] = 0.0f;
      const bool upper = h0 + 4 < HP;
#pragma unroll 4
      for (int g = 0; g < H; ++g) {
        const float p = sP[g * kKeys + key];
        const float4 lo = *reinterpret_cast<const float4*>(sT + g * HP + h0);
        w[0] = fmaf(lo.x, p, w[0]);
        w[1] = fmaf(lo.y, p, w[1]);
        w[2] = fmaf(lo.z, p, w[2]);
        w[3] = fmaf(lo.w, p, w[3]);
        if (upper) {
          const float4 hi = *reinterpret_cast<const float4*>(sT + g * HP + h0 + 4);
          w[4] = fmaf(hi.x, p, w[4]);
          w[5] = fmaf(hi.y, p, w[5]);
          w[6] = fmaf(hi.z, p, w[6]);
          w[7] = fmaf(hi.w, p, w[7]);
        }
      }
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(t.weights) + (row + h0) * t.pitch + k0 + key;
#pragma unroll
      for (int i = 0; i < kMixHeads; ++i)
        if (h0 + i < H) out[static_cast<int64_t>(i) * t.pitch] = __float2bfloat16_rn(w[i]);
    }
    __syncthreads();
  }
}

// ------------------------------------------------------------------------------------------------
// values: grid (tiles, kv_heads * head tiles, splits); MT * 16 rows, a warp takes DP / 4 value columns
// ------------------------------------------------------------------------------------------------
template <int DP, int MT>
__global__ void __launch_bounds__(kThreads)
talk_values_kernel(const NxTalkPagedArgs t, int rt, int tq, int head_tiles) {
  constexpr int LD = DP + 8, LW = kKeys + 8, COLS = DP / 4, R = MT * 16;
  const NxPagedWindowArgs& a = t.base;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* sV = sm;                       // [2 stages][64][LD]
  __nv_bfloat16* sW = sV + 2 * kKeys * LD;      // [2 stages][R][LW]
  __shared__ int s_tile[3];
  const Tile tile = locate(a.seg, tq, blockIdx.x, s_tile);
  if (!tile.ok) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hk = blockIdx.y / head_tiles, ht = blockIdx.y % head_tiles;
  const int rep = a.heads / a.kv_heads, h0 = hk * rep + ht * rt, nh = min(rt, rep - ht * rt);
  const int pos0 = a.seg.pos[tile.sg] + tile.t0;
  const int64_t row0 = static_cast<int64_t>(a.seg.row0[tile.sg]) + tile.t0, scratch0 = static_cast<int64_t>(blockIdx.x) * tq;
  const KvSource src(a, a.seg.seq[tile.sg], hk, hk);
  const KeyRange keys(a, pos0, pos0 + tile.nt - 1);
  int first, last;
  key_span(a, keys, blockIdx.z, first, last);
  const __nv_bfloat16* weights = static_cast<const __nv_bfloat16*>(t.weights);
  auto stage = [&](int k0, int s) {
    stage_rows<DP>(sV + s * kKeys * LD, src.v, src.v_pitch, a.vdim, src, keys, k0, last);
    for (int i = threadIdx.x; i < R * (kKeys / 8); i += kThreads) {
      const int m = i / (kKeys / 8), c = (i % (kKeys / 8)) * 8, tok = m / rt, hh = m % rt;
      __nv_bfloat16* d = sW + (s * R + m) * LW + c;
      if (tok < tile.nt && hh < nh) cp_async16(d, weights + ((scratch0 + tok) * a.heads + h0 + hh) * t.pitch + k0 + c);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
    }
    cp_async_commit();
  };
  if (first <= last) stage(first, 0);
  float o[MT][COLS / 8][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int n = 0; n < COLS / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[mt][n][e] = 0.0f;
  int s = 0;
  for (int k0 = first; k0 <= last; k0 += kKeys, s ^= 1) {
    if (k0 + kKeys <= last) {
      stage(k0 + kKeys, s ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const __nv_bfloat16* sv = sV + s * kKeys * LD + warp * COLS;
    const __nv_bfloat16* sw = sW + s * R * LW;
#pragma unroll
    for (int kk = 0; kk < kKeys / 16; ++kk) {
      uint32_t wa[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) ldmatrix_x4(wa[mt], smem_addr(sw + (mt * 16 + (lane & 15)) * LW + kk * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int n = 0; n < COLS / 16; ++n) {
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, smem_addr(sv + (kk * 16 + (lane & 15)) * LD + n * 16 + (lane >> 4) * 8));
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16(o[mt][2 * n], wa[mt], vb[0], vb[1]);
          mma_bf16(o[mt][2 * n + 1], wa[mt], vb[2], vb[3]);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int m = mt * 16 + i * 8 + (lane >> 2), tok = m / rt, hh = m % rt;
      if (tok >= tile.nt || hh >= nh) continue;
      const int h = h0 + hh;
      const int64_t row = row0 + tok;
      const float g = a.splits == 1 ? a.out_scale * (a.gate != nullptr ? a.gate[row * a.heads + h] : 1.0f) : 1.0f;
#pragma unroll
      for (int n = 0; n < COLS / 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int d = warp * COLS + n * 8 + (lane & 3) * 2 + e;
          if (d >= a.vdim) continue;
          const float v = o[mt][n][2 * i + e] * g;
          if (a.splits == 1)
            static_cast<__nv_bfloat16*>(a.out)[row * a.ldo + static_cast<int64_t>(h) * a.vdim + d] = __float2bfloat16_rn(v);
          else
            a.part_o[(((scratch0 + tok) * a.heads + h) * a.splits + blockIdx.z) * a.vdim + d] = v;
        }
    }
}

// the weights are normalised: the spans' products are added up
__global__ void talk_sum_kernel(const NxPagedWindowArgs a, int tq) {
  __shared__ int s_tile[3];
  const Tile tile = locate(a.seg, tq, blockIdx.x / tq, s_tile);
  const int tok = blockIdx.x % tq, h = blockIdx.y;
  if (!tile.ok || tok >= tile.nt) return;
  const int64_t row = static_cast<int64_t>(a.seg.row0[tile.sg]) + tile.t0 + tok;
  const float g = a.out_scale * (a.gate != nullptr ? a.gate[row * a.heads + h] : 1.0f);
  const float* p = a.part_o + (static_cast<int64_t>(blockIdx.x) * a.heads + h) * a.splits * a.vdim;
  for (int d = threadIdx.x; d < a.vdim; d += blockDim.x) {
    float v = 0.0f;
    for (int s = 0; s < a.splits; ++s) v += p[static_cast<int64_t>(s) * a.vdim + d];
    static_cast<__nv_bfloat16*>(a.out)[row * a.ldo + static_cast<int64_t>(h) * a.vdim + d] = __float2bfloat16_rn(v * g);
  }
}

template <typename Kernel>
int launch(Kernel kernel, const NxTalkPagedArgs* t, dim3 grid, int smem, int rt, int tq, int head_tiles, cudaStream_t st) {
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
  kernel<<<grid, kThreads, smem, st>>>(*t, rt, tq, head_tiles);
  return launch_status();
}
template <int DP, int MT>
int launch_scores(const NxTalkPagedArgs* t, dim3 grid, int rt, int tq, int head_tiles, cudaStream_t st) {
  return launch(talk_scores_kernel<DP, MT>, t, grid, (MT * 16 + 2 * kKeys) * (DP + 8) * 2, rt, tq, head_tiles, st);
}
template <int DP, int MT>
int launch_values(const NxTalkPagedArgs* t, dim3 grid, int rt, int tq, int head_tiles, cudaStream_t st) {
  return launch(talk_values_kernel<DP, MT>, t, grid, 2 * (kKeys * (DP + 8) + MT * 16 * (kKeys + 8)) * 2, rt, tq, head_tiles, st);
}
template <int MT>
int launch_all(const NxTalkPagedArgs* t, int rt, int tq, cudaStream_t st) {
  const NxPagedWindowArgs& a = t->base;
  const int head_tiles = (a.heads / a.kv_heads + rt - 1) / rt, tiles = t->rows / tq;
  const dim3 grid(tiles, a.kv_heads * head_tiles, a.splits);
  int rc = a.dim <= 64    ? launch_scores<64, MT>(t, grid, rt, tq, head_tiles, st)
           : a.dim <= 128 ? launch_scores<128, MT>(t, grid, rt, tq, head_tiles, st)
                          : launch_scores<256, MT>(t, grid, rt, tq, head_tiles, st);
  if (rc) return rc;
  const int smem = a.heads * (((a.heads + 3) & ~3) + kKeys + 1) * static_cast<int>(sizeof(float));
  if (smem > 40 * 1024 &&
      cudaFuncSetAttribute(talk_mix_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
    return -2;
  const int strides = static_cast<int>(std::max<int64_t>(1, std::min<int64_t>(t->pitch / kKeys, 4736 / std::max(1, t->rows))));
  talk_mix_kernel<<<dim3(t->rows, strides), kMixThreads, smem, st>>>(*t, tq);
  if ((rc = launch_status())) return rc;
  rc = a.vdim <= 64    ? launch_values<64, MT>(t, grid, rt, tq, head_tiles, st)
       : a.vdim <= 128 ? launch_values<128, MT>(t, grid, rt, tq, head_tiles, st)
                       : launch_values<256, MT>(t, grid, rt, tq, head_tiles, st);
  if (rc == 0 && a.splits > 1) {
    talk_sum_kernel<<<dim3(t->rows, a.heads), std::min(256, (a.vdim + 31) / 32 * 32), 0, st>>>(a, tq);
    rc = launch_status();
  }
  return rc;
}

// rows (a multiple of 16) and tokens of a tile
int tile_rows(int heads, int kv_heads, int max_len) {
  const int rt = std::min(heads / kv_heads, 16);
  return max_len == 1 ? 16 : max_len * rt <= 32 ? 32 : 64;
}
int tile_tokens(int heads, int kv_heads, int max_len) {
  return max_len == 1 ? 1 : tile_rows(heads, kv_heads, max_len) / std::min(heads / kv_heads, 16);
}

}  // namespace

extern "C" int nx_talk_rows(int heads, int kv_heads, int count, int max_len, int total_len) {
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || count <= 0 || max_len <= 0) return 0;
  const int tq = tile_tokens(heads, kv_heads, max_len);
  return max_len == 1 ? count : (total_len / tq + count) * tq;
}

extern "C" int nx_talk_paged(const NxTalkPagedArgs* t, nx_stream_t stream) {
  if (t == nullptr || t->talk == nullptr || t->scores == nullptr || t->weights == nullptr || t->pitch <= 0 || t->pitch % kKeys) return -1;
  const NxPagedWindowArgs* a = &t->base;
  if (a->dtype != NX_BF16 || a->heads <= 0 || a->heads > 96 || a->kv_heads <= 0 || a->heads % a->kv_heads) return -1;
  if (a->dim <= 0 || a->dim > 256 || a->vdim <= 0 || a->vdim > 256 || a->block_size <= 0 || a->max_blocks <= 0) return -1;
  if (a->splits < 1 || a->splits > 65535 || a->part_ml == nullptr || (a->splits > 1 && a->part_o == nullptr)) return -1;
  if (a->sink != nullptr || a->all_values || a->keep_first < 0 || a->chunk < 0 || (a->bias != nullptr && a->bias_len <= 0)) return -1;
  if (a->k_pitch < static_cast<int64_t>(a->kv_heads) * a->dim || a->v_pitch < static_cast<int64_t>(a->kv_heads) * a->vdim) return -1;
  if ((reinterpret_cast<uintptr_t>(t->scores) | reinterpret_cast<uintptr_t>(t->weights)) & 15) return -1;
  if (a->seg.count <= 0 || a->seg.max_len <= 0) return 0;
  if (t->rows != nx_talk_rows(a->heads, a->kv_heads, a->seg.count, a->seg.max_len, a->seg.total_len)) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int rt = std::min(a->heads / a->kv_heads, 16), tq = tile_tokens(a->heads, a->kv_heads, a->seg.max_len);
  switch (tile_rows(a->heads, a->kv_heads, a->seg.max_len)) {
    case 16: return launch_all<1>(t, rt, tq, st);
    case 32: return launch_all<2>(t, rt, tq, st);
    default: return launch_all<4>(t, rt, tq, st);
  }
}
