// Chunked tensor-core forms of the two recurrences (see nx_api_mixers.h) for long segments with BF16 activations.  A chunk
// is 64 tokens; a block carries the FP32 state of one head (one tile of value columns of it) through the chunks of its
// segment in registers, as the accumulators of the products that update it.
//
// Precision: projections and convolution outputs are BF16 and enter the products as they are; everything derived from
// decays, step sizes and the state is FP32, and where such a value has to be an operand it is split into a BF16 pair
// (value and rounding remainder) that is multiplied in two products, which keeps 16 bits of mantissa.  Unit vectors are
// never rounded: their inverse norms scale the FP32 results of products of the raw vectors.
//
// State-space chunk, a_t = log decay of token t, c_t = a_1 + .. + a_t, S the incoming state:
//   y_t = e^{c_t} S^T C_t + sum_{s <= t} e^{c_t - c_s} dt_s (C_t . B_s) x_s + D x_t
//   S'  = e^{c_Q} S + sum_s B_s (e^{c_Q - c_s} dt_s x_s)^T
// Delta-rule chunk, b_t = cumulative log decay, k / q unit vectors:
//   (I + A) U = R,  A_ts = beta_t e^{b_t - b_s} (k_t . k_s) for s < t,  R_t = beta_t (v_t - e^{b_t} S^T k_t)
//   o_t = e^{b_t} S^T q_t + sum_{s <= t} e^{b_t - b_s} (k_s . q_t) U_s
//   S'  = e^{b_Q} S + sum_s k_s (e^{b_Q - b_s} U_s)^T
// (I + A)^{-1} and the masked q k products do not depend on the state: a first kernel forms them for all chunks at once.
#include "mixer_common.cuh"
#include "nx_api_mixers.h"

#include <algorithm>

namespace {
using namespace nx;

constexpr int kQ = 64;                 // tokens per chunk
constexpr int kCols = 64;              // value columns per block (state-space)
constexpr float kLog2e = 1.4426950408889634f;

// rows x cols BF16 of a row-major matrix into shared memory [64][LD]; rows past `rows` and columns past `cols` (up to PAD)
// are zeros.  `vec`: 16-byte copies are possible.
template <int PAD>
__device__ __forceinline__ void load_tile(__nv_bfloat16* dst, const __nv_bfloat16* src, int64_t ld, int rows, int cols, bool vec) {
  constexpr int LD = PAD + 8, CH = PAD / 8;
  for (int i = threadIdx.x; i < kQ * CH; i += blockDim.x) {
    const int r = i / CH, c = (i % CH) * 8;
    __nv_bfloat16* d = dst + r * LD + c;
    if (r < rows && c < cols) {
      const __nv_bfloat16* s = src + r * ld + c;
      if (vec) {
        cp_async16(d, s);
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) d[e] = c + e < cols ? s[e] : __float2bfloat16_rn(0.0f);
      }
    } else {
      *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
    }
  }
}

// fragment addresses inside a [rows][LD] BF16 tile
template <int LD>
__device__ __forceinline__ uint32_t addr_a(const __nv_bfloat16* t, int row, int col) {       // A, row-major
  const int lane = threadIdx.x & 31;
  return smem_addr(t + (row + (lane & 15)) * LD + col + (lane >> 4) * 8);
}
template <int LD>
__device__ __forceinline__ uint32_t addr_a_t(const __nv_bfloat16* t, int k, int m) {         // A = transpose of the tile
  const int lane = threadIdx.x & 31;
  return smem_addr(t + (k + ((lane >> 4) << 3) + (lane & 7)) * LD + m + ((lane >> 3) & 1) * 8);
}
template <int LD>
__device__ __forceinline__ uint32_t addr_b(const __nv_bfloat16* t, int n, int k) {           // B[k][n] = tile[n][k]
  const int lane = threadIdx.x & 31;
  return smem_addr(t + (n + (lane & 7) + ((lane >> 4) << 3)) * LD + k + ((lane >> 3) & 1) * 8);
}
template <int LD>
__device__ __forceinline__ uint32_t addr_b_t(const __nv_bfloat16* t, int k, int n) {         // B[k][n] = tile[k][n]
  const int lane = threadIdx.x & 31;
  return smem_addr(t + (k + (lane & 15)) * LD + n + (lane >> 4) * 8);
}

template <int N>
__device__ __forceinline__ void zero(float (&d)[N][4]) {
#pragma unroll
  for (int i = 0; i < N; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) d[i][e] = 0.0f;
}

// an FP32 accumulator tile (16 rows x 8 NT columns) as a pair of BF16 tiles in shared memory
template <int NT, int LD>
__device__ __forceinline__ void store_split(__nv_bfloat16* hi, __nv_bfloat16* lo, int row, const float (&v)[NT][4]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      uint32_t h, l;
      bf16_split(v[n][2 * i], v[n][2 * i + 1], h, l);
      const int o = (row + i * 8 + (lane >> 2)) * LD + n * 8 + (lane & 3) * 2;
      *reinterpret_cast<uint32_t*>(hi + o) = h;
      *reinterpret_cast<uint32_t*>(lo + o) = l;
    }
}

// inclusive sums of 64 values held two per lane (elements lane and lane + 32) by one warp
__device__ __forceinline__ void scan64(float& v0, float& v1) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float a = __shfl_up_sync(0xffffffffu, v0, o), b = __shfl_up_sync(0xffffffffu, v1, o);
    if (lane >= o) {
      v0 += a;
      v1 += b;
    }
  }
  v1 += __shfl_sync(0xffffffffu, v0, 31);
}

// ------------------------------------------------------------------------------------------------
// state-space duality.  grid (heads * column tiles, parts, segments), 4 warps.  Warp w owns token rows
// 16 w .. 16 w + 15 of the chunk's outputs and NP / 4 rows of the state.
// kLocal: only the span's own contribution to the state, from zero, and its decay (for spans that run
// at the same time); otherwise outputs, from the span's true start state.
// ------------------------------------------------------------------------------------------------
template <int NP>
struct SsdSmem {
  static constexpr int LN = NP + 8, LP = kCols + 8;
  static constexpr int kB = 0, kC = kB + kQ * LN, kX = kC + kQ * LN, kXh = kX + kQ * LP, kXl = kXh + kQ * LP,
                       kSh = kXl + kQ * LP, kSl = kSh + NP * LP, kEnd = kSl + NP * LP;
  static constexpr int kBytes = kEnd * 2;
};

template <int NP, bool kLocal>
__global__ void __launch_bounds__(128) ssd_chunk_kernel(const NxSsdArgs a, int col_tiles) {
  using L = SsdSmem<NP>;
  constexpr int LN = L::LN, LP = L::LP, MT = NP / 64;    // MT: 16-row tiles of the state per warp
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16 *sB = sm + L::kB, *sC = sm + L::kC, *sX = sm + L::kX, *sXh = sm + L::kXh, *sXl = sm + L::kXl,
                *sSh = sm + L::kSh, *sSl = sm + L::kSl;
  __shared__ float s_c[kQ], s_dt[kQ];                    // cumulative log2 decay, step size
  const int h = blockIdx.x / col_tiles, p0 = (blockIdx.x % col_tiles) * kCols, part = blockIdx.y, sg = blockIdx.z;
  const int len = a.seg.len[sg], t_begin = part * a.span, t_end = min(len, t_begin + a.span);
  if (t_begin >= len || (kLocal && t_end == len)) return;   // the last span's contribution is never needed
  const int N = a.n_state, P = a.vdim, cols = min(kCols, P - p0), inner = a.heads * P, g = h / (a.heads / a.groups);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, qr = lane >> 2, qc = (lane & 3) * 2;
  const int64_t row0 = a.seg.row0[sg];
  const __nv_bfloat16* xbc = static_cast<const __nv_bfloat16*>(a.xbc) + row0 * a.ld_xbc;
  const __nv_bfloat16* dtp = static_cast<const __nv_bfloat16*>(a.dt) + row0 * a.ld_dt + h;
  const bool aligned = (a.ld_xbc & 7) == 0 && (inner & 7) == 0 && (reinterpret_cast<uintptr_t>(a.xbc) & 15) == 0;
  const bool vec_n = aligned && (N & 7) == 0, vec_p = aligned && (P & 7) == 0;
  const float rate = -expf(a.a_log[h]) * kLog2e, dtb = a.dt_bias[h], skip = a.d_skip[h];
  const int64_t plane = static_cast<int64_t>(N) * P;
  float* pool = a.state + (static_cast<int64_t>(a.seg.seq[sg]) * a.heads + h) * plane;
  float* part_state = a.parts > 1 ? a.part_state + ((static_cast<int64_t>(sg) * a.parts + part) * a.heads + h) * plane : nullptr;
  float S[MT][8][4];
  {
    const float* src = kLocal ? nullptr : a.parts > 1 ? part_state : (a.seg.pos[sg] == 0 ? nullptr : pool);
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = (warp * MT + m) * 16 + (e >> 1) * 8 + qr, c = n * 8 + qc + (e & 1);
          S[m][n][e] = (src != nullptr && r < N && c < cols) ? src[static_cast<int64_t>(r) * P + p0 + c] : 0.0f;
        }
  }
  float total = 0.0f;                                    // log2 decay of the whole span
  for (int t0 = t_begin; t0 < t_end; t0 += kQ) {
    const int rows = min(kQ, t_end - t0);
    const __nv_bfloat16* src = xbc + t0 * a.ld_xbc;
    load_tile<NP>(sB, src + inner + g * N, a.ld_xbc, rows, N, vec_n);
    if (!kLocal) load_tile<NP>(sC, src + inner + (a.groups + g) * N, a.ld_xbc, rows, N, vec_n);
    load_tile<kCols>(sX, src + h * P + p0, a.ld_xbc, rows, cols, vec_p);
    cp_async_commit();
    if (warp == 0) {
      float d[2], c[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = lane + 32 * i;
        d[i] = t < rows ? softplus_exact(__bfloat162float(dtp[(t0 + t) * a.ld_dt]) + dtb) : 0.0f;
        c[i] = rate * d[i];
      }
      scan64(c[0], c[1]);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        s_dt[lane + 32 * i] = d[i];
        s_c[lane + 32 * i] = c[i];
      }
    }
    if (!kLocal) {
#pragma unroll
      for (int m = 0; m < MT; ++m) store_split<8, LP>(sSh, sSl, (warp * MT + m) * 16, S[m]);
    }
    cp_async_wait<0>();
    __syncthreads();
    const float c_end = s_c[kQ - 1];
    // x weighted for the state update
    for (int i = threadIdx.x; i < kQ * (kCols / 2); i += 128) {
      const int t = i / (kCols / 2), o = t * LP + (i % (kCols / 2)) * 2;
      const float w = exp2f(c_end - s_c[t]) * s_dt[t];
      const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(sX + o);
      uint32_t hi, lo;
      bf16_split(__low2float(x) * w, __high2float(x) * w, hi, lo);
      *reinterpret_cast<uint32_t*>(sXh + o) = hi;
      *reinterpret_cast<uint32_t*>(sXl + o) = lo;
    }
    if (!kLocal) {
      const float ci[2] = {s_c[warp * 16 + qr], s_c[warp * 16 + 8 + qr]};
      float y[8][4];
      zero(y);
#pragma unroll
      for (int kk = 0; kk < NP / 16; ++kk) {             // C S
        uint32_t ca[4];
        ldmatrix_x4(ca, addr_a<LN>(sC, warp * 16, kk * 16));
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, addr_b_t<LP>(sSh, kk * 16, n * 16));
          mma_bf16(y[2 * n], ca, b[0], b[1]);
          mma_bf16(y[2 * n + 1], ca, b[2], b[3]);
          ldmatrix_x4_trans(b, addr_b_t<LP>(sSl, kk * 16, n * 16));
          mma_bf16(y[2 * n], ca, b[0], b[1]);
          mma_bf16(y[2 * n + 1], ca, b[2], b[3]);
        }
      }
      const float e0 = exp2f(ci[0]), e1 = exp2f(ci[1]);
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        y[n][0] *= e0;
        y[n][1] *= e0;
        y[n][2] *= e1;
        y[n][3] *= e1;
      }
      for (int j = 0; j <= warp; ++j) {                  // 16 keys at a time, up to the diagonal
        float gm[2][4];
        zero(gm);
#pragma unroll
        for (int kk = 0; kk < NP / 16; ++kk) {
          uint32_t ca[4], b[4];
          ldmatrix_x4(ca, addr_a<LN>(sC, warp * 16, kk * 16));
          ldmatrix_x4(b, addr_b<LN>(sB, j * 16, kk * 16));
          mma_bf16(gm[0], ca, b[0], b[1]);
          mma_bf16(gm[1], ca, b[2], b[3]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int s = j * 16 + n * 8 + qc + (e & 1), t = warp * 16 + (e >> 1) * 8 + qr;
            gm[n][e] = s <= t ? gm[n][e] * exp2f(ci[e >> 1] - s_c[s]) * s_dt[s] : 0.0f;
          }
        uint32_t mh[4], ml[4];
        bf16_split(gm[0][0], gm[0][1], mh[0], ml[0]);
        bf16_split(gm[0][2], gm[0][3], mh[1], ml[1]);
        bf16_split(gm[1][0], gm[1][1], mh[2], ml[2]);
        bf16_split(gm[1][2], gm[1][3], mh[3], ml[3]);
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, addr_b_t<LP>(sX, j * 16, n * 16));
          mma_bf16(y[2 * n], mh, b[0], b[1]);
          mma_bf16(y[2 * n + 1], mh, b[2], b[3]);
          mma_bf16(y[2 * n], ml, b[0], b[1]);
          mma_bf16(y[2 * n + 1], ml, b[2], b[3]);
        }
      }
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.y) + (row0 + t0) * a.ldy + static_cast<int64_t>(h) * P + p0;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = warp * 16 + i * 8 + qr;
        if (t >= rows) continue;
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          const int c = n * 8 + qc;
          const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(sX + t * LP + c);
          const float v0 = y[n][2 * i] + skip * __low2float(x), v1 = y[n][2 * i + 1] + skip * __high2float(x);
          if (c < cols) out[t * a.ldy + c] = __float2bfloat16_rn(v0);
          if (c + 1 < cols) out[t * a.ldy + c + 1] = __float2bfloat16_rn(v1);
        }
      }
    }
    __syncthreads();                                     // weighted x complete
    const float dec = exp2f(c_end);
    total += c_end;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][n][e] *= dec;
#pragma unroll
    for (int kk = 0; kk < kQ / 16; ++kk) {
      uint32_t ba[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldmatrix_x4_trans(ba[m], addr_a_t<LN>(sB, kk * 16, (warp * MT + m) * 16));
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bh, addr_b_t<LP>(sXh, kk * 16, n * 16));
        ldmatrix_x4_trans(bl, addr_b_t<LP>(sXl, kk * 16, n * 16));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16(S[m][2 * n], ba[m], bh[0], bh[1]);
          mma_bf16(S[m][2 * n + 1], ba[m], bh[2], bh[3]);
          mma_bf16(S[m][2 * n], ba[m], bl[0], bl[1]);
          mma_bf16(S[m][2 * n + 1], ba[m], bl[2], bl[3]);
        }
      }
    }
    __syncthreads();                                     // before the tiles are loaded over
  }
  float* dst = kLocal ? part_state : (t_end == len ? pool : nullptr);
  if (dst != nullptr) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = (warp * MT + m) * 16 + (e >> 1) * 8 + qr, c = n * 8 + qc + (e & 1);
          if (r < N && c < cols) dst[static_cast<int64_t>(r) * P + p0 + c] = S[m][n][e];
        }
    if (kLocal && threadIdx.x == 0 && p0 == 0)
      a.part_decay[(static_cast<int64_t>(sg) * a.parts + part) * a.heads + h] = exp2f(total);
  }
}

// start state of every span from the spans' own contributions: grid (heads, segments, element blocks)
__global__ void ssd_span_scan_kernel(const NxSsdArgs a) {
  const int h = blockIdx.x, sg = blockIdx.y;
  const int64_t plane = static_cast<int64_t>(a.n_state) * a.vdim;
  const int64_t i = blockIdx.z * static_cast<int64_t>(blockDim.x) + threadIdx.x;
  if (i >= plane) return;
  const int len = a.seg.len[sg];
  float s = a.seg.pos[sg] == 0 ? 0.0f : a.state[(static_cast<int64_t>(a.seg.seq[sg]) * a.heads + h) * plane + i];
  for (int k = 0; k * a.span < len; ++k) {
    const int64_t idx = (static_cast<int64_t>(sg) * a.parts + k) * a.heads + h;
    float* p = a.part_state + idx * plane + i;
    const bool last = (k + 1) * a.span >= len;
    const float own = last ? 0.0f : *p;
    *p = s;
    if (!last) s = a.part_decay[idx] * s + own;
  }
}

template <int NP>
int launch_ssd(const NxSsdArgs* a, cudaStream_t st) {
  constexpr int kBytes = SsdSmem<NP>::kBytes;
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(ssd_chunk_kernel<NP, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes) != cudaSuccess ||
        cudaFuncSetAttribute(ssd_chunk_kernel<NP, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes) != cudaSuccess)
      return -2;
    once = true;
  }
  const int col_tiles = (a->vdim + kCols - 1) / kCols;
  dim3 grid(a->heads * col_tiles, a->parts, a->seg.count);
  if (a->parts > 1) {
    ssd_chunk_kernel<NP, true><<<grid, 128, kBytes, st>>>(*a, col_tiles);
    const int plane = a->n_state * a->vdim;
    ssd_span_scan_kernel<<<dim3(a->heads, a->seg.count, (plane + 255) / 256), 256, 0, st>>>(*a);
  }
  ssd_chunk_kernel<NP, false><<<grid, 128, kBytes, st>>>(*a, col_tiles);
  return launch_status();
}

// ------------------------------------------------------------------------------------------------
// delta rule, first kernel: everything of a chunk that does not depend on the state.
// grid (chunks, heads, segments), 4 warps.  Scratch per (segment, chunk, head): T hi | T lo | P hi | P lo, each [64][64]
// BF16, then FP32 [4][64]: cumulative log2 decay, 1 / |k|, dim^-1/2 / |q|, beta.
// ------------------------------------------------------------------------------------------------
constexpr int64_t kDeltaTile = kQ * kQ;
constexpr int64_t kDeltaUnit = 4 * kDeltaTile + 4 * kQ * 2;   // in BF16 elements

template <int DP>
__global__ void __launch_bounds__(128) delta_prep_kernel(const NxDeltaArgs a, int chunks) {
  constexpr int LD = DP + 8, LA = kQ + 4;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16 *sK = sm, *sQ = sm + kQ * LD;
  float* sA = reinterpret_cast<float*>(sm + 2 * kQ * LD);     // [64][LA]
  __shared__ float s_b[kQ], s_rk[kQ], s_rq[kQ], s_beta[kQ];
  const int ch = blockIdx.x, h = blockIdx.y, sg = blockIdx.z, t0 = ch * kQ;
  const int len = a.seg.len[sg];
  if (t0 >= len) return;
  const int rows = min(kQ, len - t0), D = a.dim, hk = h / (a.heads / a.kv_heads), kcols = a.kv_heads * D;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, qr = lane >> 2, qc = (lane & 3) * 2;
  const int64_t row0 = static_cast<int64_t>(a.seg.row0[sg]) + t0;
  const __nv_bfloat16* qkv = static_cast<const __nv_bfloat16*>(a.qkv) + row0 * a.ld_qkv;
  const bool vec = (a.ld_qkv & 7) == 0 && (D & 7) == 0 && (reinterpret_cast<uintptr_t>(a.qkv) & 15) == 0;
  load_tile<DP>(sQ, qkv + hk * D, a.ld_qkv, rows, D, vec);
  load_tile<DP>(sK, qkv + kcols + hk * D, a.ld_qkv, rows, D, vec);
  cp_async_commit();
  if (warp == 0) {
    const float rate = -expf(a.a_log[h]) * kLog2e, dtb = a.dt_bias[h];
    float g[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = lane + 32 * i;
      g[i] = 0.0f;
      float beta = 0.0f;
      if (t < rows) {
        const int64_t o = (row0 + t) * a.ld_ba + h;
        g[i] = rate * softplus_exact(__bfloat162float(static_cast<const __nv_bfloat16*>(a.a)[o]) + dtb);
        beta = sigmoid_exact(__bfloat162float(static_cast<const __nv_bfloat16*>(a.b)[o]));
      }
      s_beta[t] = beta;
    }
    scan64(g[0], g[1]);
    s_b[lane] = g[0];
    s_b[lane + 32] = g[1];
  }
  cp_async_wait<0>();
  __syncthreads();
  {                                            // inverse norms: two threads per row
    const int t = threadIdx.x >> 1, half = threadIdx.x & 1;
    float kk = 0.0f, qq = 0.0f;
    for (int d = half * 2; d < DP; d += 4) {
      const __nv_bfloat162 k = *reinterpret_cast<const __nv_bfloat162*>(sK + t * LD + d);
      const __nv_bfloat162 q = *reinterpret_cast<const __nv_bfloat162*>(sQ + t * LD + d);
      kk += __low2float(k) * __low2float(k) + __high2float(k) * __high2float(k);
      qq += __low2float(q) * __low2float(q) + __high2float(q) * __high2float(q);
    }
    kk += __shfl_xor_sync(0xffffffffu, kk, 1);
    qq += __shfl_xor_sync(0xffffffffu, qq, 1);
    if (half == 0) {
      s_rk[t] = 1.0f / sqrtf(kk + a.unit_eps);
      s_rq[t] = a.q_scale / sqrtf(qq + a.unit_eps);
    }
  }
  __syncthreads();
  __nv_bfloat16* unit = static_cast<__nv_bfloat16*>(a.scratch) +
                        ((static_cast<int64_t>(sg) * chunks + ch) * a.heads + h) * kDeltaUnit;
  __nv_bfloat16 *Th = unit, *Tl = unit + kDeltaTile, *Ph = unit + 2 * kDeltaTile, *Pl = unit + 3 * kDeltaTile;
  const float bt[2] = {s_b[warp * 16 + qr], s_b[warp * 16 + 8 + qr]};
  const float rkt[2] = {s_rk[warp * 16 + qr], s_rk[warp * 16 + 8 + qr]};
  const float rqt[2] = {s_rq[warp * 16 + qr], s_rq[warp * 16 + 8 + qr]};
  const float bet[2] = {s_beta[warp * 16 + qr], s_beta[warp * 16 + 8 + qr]};
#pragma unroll
  for (int j = 0; j < kQ / 16; ++j) {
    float kk[2][4], qk[2][4];
    zero(kk);
    zero(qk);
    if (j <= warp) {
#pragma unroll
      for (int d = 0; d < DP / 16; ++d) {
        uint32_t ka[4], qa[4], b[4];
        ldmatrix_x4(ka, addr_a<LD>(sK, warp * 16, d * 16));
        ldmatrix_x4(qa, addr_a<LD>(sQ, warp * 16, d * 16));
        ldmatrix_x4(b, addr_b<LD>(sK, j * 16, d * 16));
        mma_bf16(kk[0], ka, b[0], b[1]);
        mma_bf16(kk[1], ka, b[2], b[3]);
        mma_bf16(qk[0], qa, b[0], b[1]);
        mma_bf16(qk[1], qa, b[2], b[3]);
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = warp * 16 + i * 8 + qr, s = j * 16 + n * 8 + qc;
        float p[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float w = s + e <= t ? exp2f(bt[i] - s_b[s + e]) * s_rk[s + e] : 0.0f;
          p[e] = qk[n][2 * i + e] * w * rqt[i];
          sA[t * LA + s + e] = s + e < t ? kk[n][2 * i + e] * w * rkt[i] * bet[i] : 0.0f;
        }
        uint32_t hi, lo;
        bf16_split(p[0], p[1], hi, lo);
        *reinterpret_cast<uint32_t*>(Ph + t * kQ + s) = hi;
        *reinterpret_cast<uint32_t*>(Pl + t * kQ + s) = lo;
      }
  }
  __syncthreads();
  if (threadIdx.x < kQ) {                      // column c of (I + A)^-1 by forward substitution, in registers
    const int c = threadIdx.x;
    float x[kQ];
#pragma unroll
    for (int i = 0; i < kQ; ++i) {
      float v0 = i == c ? 1.0f : 0.0f, v1 = 0.0f, v2 = 0.0f, v3 = 0.0f;
#pragma unroll
      for (int j = 0; j + 3 < i; j += 4) {
        const float4 r = *reinterpret_cast<const float4*>(sA + i * LA + j);
        v0 -= r.x * x[j];
        v1 -= r.y * x[j + 1];
        v2 -= r.z * x[j + 2];
        v3 -= r.w * x[j + 3];
      }
#pragma unroll
      for (int j = i / 4 * 4; j < i; ++j) v0 -= sA[i * LA + j] * x[j];
      x[i] = (v0 + v1) + (v2 + v3);
    }
#pragma unroll
    for (int i = 0; i < kQ; ++i) {
      const __nv_bfloat16 hi = __float2bfloat16_rn(x[i]);
      Th[i * kQ + c] = hi;
      Tl[i * kQ + c] = __float2bfloat16_rn(x[i] - __bfloat162float(hi));
    }
    float* sc = reinterpret_cast<float*>(unit + 4 * kDeltaTile);
    sc[c] = s_b[c];
    sc[kQ + c] = s_rk[c];
    sc[2 * kQ + c] = s_rq[c];
    sc[3 * kQ + c] = s_beta[c];
  }
}

// ------------------------------------------------------------------------------------------------
// delta rule, second kernel: the chunks of a segment in order.  grid (heads * column tiles, segments),
// 4 warps; warp w owns token rows 16 w .. of U and the outputs, and DP / 4 rows of the state.
// ------------------------------------------------------------------------------------------------
constexpr int kDeltaCols = 32;

template <int DP>
struct DeltaSmem {
  static constexpr int LD = DP + 8, LV = kDeltaCols + 8, LT = kQ + 8;
  static constexpr int kK = 0, kQq = kK + kQ * LD, kV = kQq + kQ * LD, kTh = kV + kQ * LV, kTl = kTh + kQ * LT,
                       kPh = kTl + kQ * LT, kPl = kPh + kQ * LT, kRh = kPl + kQ * LT, kRl = kRh + kQ * LV, kUh = kRl + kQ * LV,
                       kUl = kUh + kQ * LV, kSh = kUl + kQ * LV, kSl = kSh + DP * LV, kEnd = kSl + DP * LV;
  static constexpr int kBytes = kEnd * 2;
};

// d += (ah + al) (bh + bl) up to the product of the two remainders, over the first `kblocks` blocks of 16
template <int LT, int LV>
__device__ __forceinline__ void mma_split(float (&d)[kDeltaCols / 8][4], const __nv_bfloat16* ah, const __nv_bfloat16* al,
                                          const __nv_bfloat16* bh, const __nv_bfloat16* bl, int row, int kblocks) {
  for (int kk = 0; kk < kblocks; ++kk) {
    uint32_t fh[4], fl[4];
    ldmatrix_x4(fh, addr_a<LT>(ah, row, kk * 16));
    ldmatrix_x4(fl, addr_a<LT>(al, row, kk * 16));
#pragma unroll
    for (int n = 0; n < kDeltaCols / 16; ++n) {
      uint32_t gh[4], gl[4];
      ldmatrix_x4_trans(gh, addr_b_t<LV>(bh, kk * 16, n * 16));
      ldmatrix_x4_trans(gl, addr_b_t<LV>(bl, kk * 16, n * 16));
      mma_bf16(d[2 * n], fh, gh[0], gh[1]);
      mma_bf16(d[2 * n + 1], fh, gh[2], gh[3]);
      mma_bf16(d[2 * n], fh, gl[0], gl[1]);
      mma_bf16(d[2 * n + 1], fh, gl[2], gl[3]);
      mma_bf16(d[2 * n], fl, gh[0], gh[1]);
      mma_bf16(d[2 * n + 1], fl, gh[2], gh[3]);
    }
  }
}

template <int DP>
__global__ void __launch_bounds__(128) delta_chunk_kernel(const NxDeltaArgs a, int chunks, int col_tiles) {
  using L = DeltaSmem<DP>;
  constexpr int LD = L::LD, LV = L::LV, LT = L::LT, MT = DP / 64, NT = kDeltaCols / 8;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16 *sK = sm + L::kK, *sQ = sm + L::kQq, *sV = sm + L::kV, *sTh = sm + L::kTh, *sTl = sm + L::kTl,
                *sPh = sm + L::kPh, *sPl = sm + L::kPl, *sRh = sm + L::kRh, *sRl = sm + L::kRl, *sUh = sm + L::kUh,
                *sUl = sm + L::kUl, *sSh = sm + L::kSh, *sSl = sm + L::kSl;
  __shared__ __align__(16) float s_sc[4 * kQ];           // cumulative log2 decay | 1/|k| | scaled 1/|q| | beta
  const int h = blockIdx.x / col_tiles, v0 = (blockIdx.x % col_tiles) * kDeltaCols, sg = blockIdx.y;
  const int len = a.seg.len[sg];
  if (len <= 0) return;
  const int D = a.dim, Dv = a.vdim, cols = min(kDeltaCols, Dv - v0), hk = h / (a.heads / a.kv_heads), kcols = a.kv_heads * D;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, qr = lane >> 2, qc = (lane & 3) * 2;
  const int64_t row0 = a.seg.row0[sg];
  const bool aligned = (a.ld_qkv & 7) == 0 && (reinterpret_cast<uintptr_t>(a.qkv) & 15) == 0;
  const bool vec_d = aligned && (D & 7) == 0, vec_v = aligned && (Dv & 7) == 0 && ((2 * kcols) & 7) == 0;
  float* pool = a.state + (static_cast<int64_t>(a.seg.seq[sg]) * a.heads + h) * D * Dv;
  const bool fresh = a.seg.pos[sg] == 0;
  float S[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = (warp * MT + m) * 16 + (e >> 1) * 8 + qr, c = n * 8 + qc + (e & 1);
        S[m][n][e] = (!fresh && r < D && c < cols) ? pool[static_cast<int64_t>(r) * Dv + v0 + c] : 0.0f;
      }
  for (int ch = 0; ch * kQ < len; ++ch) {
    const int t0 = ch * kQ, rows = min(kQ, len - t0);
    const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(a.qkv) + (row0 + t0) * a.ld_qkv;
    const __nv_bfloat16* unit = static_cast<const __nv_bfloat16*>(a.scratch) +
                                ((static_cast<int64_t>(sg) * chunks + ch) * a.heads + h) * kDeltaUnit;
    load_tile<DP>(sQ, src + hk * D, a.ld_qkv, rows, D, vec_d);
    load_tile<DP>(sK, src + kcols + hk * D, a.ld_qkv, rows, D, vec_d);
    load_tile<kDeltaCols>(sV, src + 2 * kcols + h * Dv + v0, a.ld_qkv, rows, cols, vec_v);
    for (int i = threadIdx.x; i < 4 * kQ * 8; i += 128) {       // T and P tiles, 16 bytes each
      const int m = i / (kQ * 8), r = (i / 8) % kQ, c = (i % 8) * 8;
      cp_async16(sTh + m * (kQ * LT) + r * LT + c, unit + m * kDeltaTile + r * kQ + c);
    }
    for (int i = threadIdx.x; i < kQ; i += 128)
      cp_async16(s_sc + i * 4, reinterpret_cast<const float*>(unit + 4 * kDeltaTile) + i * 4);
    cp_async_commit();
#pragma unroll
    for (int m = 0; m < MT; ++m) store_split<NT, LV>(sSh, sSl, (warp * MT + m) * 16, S[m]);
    cp_async_wait<0>();
    __syncthreads();
    const float b_end = s_sc[kQ - 1];
    float eb[2], rk[2], rq[2], beta[2], wk[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = warp * 16 + i * 8 + qr;
      eb[i] = exp2f(s_sc[t]);
      rk[i] = s_sc[kQ + t];
      rq[i] = s_sc[2 * kQ + t];
      beta[i] = s_sc[3 * kQ + t];
      wk[i] = exp2f(b_end - s_sc[t]) * rk[i];
    }
    float ks[NT][4], o[NT][4];
    zero(ks);
    zero(o);
#pragma unroll
    for (int d = 0; d < DP / 16; ++d) {
      uint32_t ka[4], qa[4];
      ldmatrix_x4(ka, addr_a<LD>(sK, warp * 16, d * 16));
      ldmatrix_x4(qa, addr_a<LD>(sQ, warp * 16, d * 16));
#pragma unroll
      for (int n = 0; n < NT / 2; ++n) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bh, addr_b_t<LV>(sSh, d * 16, n * 16));
        ldmatrix_x4_trans(bl, addr_b_t<LV>(sSl, d * 16, n * 16));
        mma_bf16(ks[2 * n], ka, bh[0], bh[1]);
        mma_bf16(ks[2 * n + 1], ka, bh[2], bh[3]);
        mma_bf16(o[2 * n], qa, bh[0], bh[1]);
        mma_bf16(o[2 * n + 1], qa, bh[2], bh[3]);
        mma_bf16(ks[2 * n], ka, bl[0], bl[1]);
        mma_bf16(ks[2 * n + 1], ka, bl[2], bl[3]);
        mma_bf16(o[2 * n], qa, bl[0], bl[1]);
        mma_bf16(o[2 * n + 1], qa, bl[2], bl[3]);
      }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = e >> 1, t = warp * 16 + i * 8 + qr;
        const float v = __bfloat162float(sV[t * LV + n * 8 + qc + (e & 1)]);
        ks[n][e] = beta[i] * (v - eb[i] * rk[i] * ks[n][e]);
        o[n][e] *= eb[i] * rq[i];
      }
    store_split<NT, LV>(sRh, sRl, warp * 16, ks);
    __syncthreads();
    float u[NT][4];
    zero(u);
    mma_split<LT, LV>(u, sTh, sTl, sRh, sRl, warp * 16, warp + 1);
    store_split<NT, LV>(sUh, sUl, warp * 16, u);
    __syncthreads();                                     // U complete, R no longer read: it takes the weighted U
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) u[n][e] *= wk[e >> 1];
    store_split<NT, LV>(sRh, sRl, warp * 16, u);
    mma_split<LT, LV>(o, sPh, sPl, sUh, sUl, warp * 16, warp + 1);
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.o) + (row0 + t0) * a.ldo + static_cast<int64_t>(h) * Dv + v0;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = warp * 16 + (e >> 1) * 8 + qr, c = n * 8 + qc + (e & 1);
        if (t < rows && c < cols) out[t * a.ldo + c] = __float2bfloat16_rn(o[n][e]);
      }
    __syncthreads();
    const float dec = exp2f(b_end);
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][n][e] *= dec;
#pragma unroll
    for (int kk = 0; kk < kQ / 16; ++kk) {
      uint32_t ka[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldmatrix_x4_trans(ka[m], addr_a_t<LD>(sK, kk * 16, (warp * MT + m) * 16));
#pragma unroll
      for (int n = 0; n < NT / 2; ++n) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bh, addr_b_t<LV>(sRh, kk * 16, n * 16));
        ldmatrix_x4_trans(bl, addr_b_t<LV>(sRl, kk * 16, n * 16));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16(S[m][2 * n], ka[m], bh[0], bh[1]);
          mma_bf16(S[m][2 * n + 1], ka[m], bh[2], bh[3]);
          mma_bf16(S[m][2 * n], ka[m], bl[0], bl[1]);
          mma_bf16(S[m][2 * n + 1], ka[m], bl[2], bl[3]);
        }
      }
    }
    __syncthreads();                                     // before the tiles are loaded over
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = (warp * MT + m) * 16 + (e >> 1) * 8 + qr, c = n * 8 + qc + (e & 1);
        if (r < D && c < cols) pool[static_cast<int64_t>(r) * Dv + v0 + c] = S[m][n][e];
      }
}

template <int DP>
int launch_delta(const NxDeltaArgs* a, cudaStream_t st) {
  constexpr int kBytes = DeltaSmem<DP>::kBytes, kPrep = 2 * kQ * (DP + 8) * 2 + kQ * (kQ + 4) * 4;
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(delta_chunk_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes) != cudaSuccess ||
        cudaFuncSetAttribute(delta_prep_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPrep) != cudaSuccess)
      return -2;
    once = true;
  }
  const int chunks = (a->seg.max_len + kQ - 1) / kQ, col_tiles = (a->vdim + kDeltaCols - 1) / kDeltaCols;
  delta_prep_kernel<DP><<<dim3(chunks, a->heads, a->seg.count), 128, kPrep, st>>>(*a, chunks);
  delta_chunk_kernel<DP><<<dim3(a->heads * col_tiles, a->seg.count), 128, kBytes, st>>>(*a, chunks, col_tiles);
  return launch_status();
}

}  // namespace

extern "C" int nx_ssd_chunk(const NxSsdArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->dtype != NX_BF16 || a->heads <= 0 || a->groups <= 0 || a->heads % a->groups) return -1;
  if (a->n_state <= 0 || a->vdim <= 0 || a->parts < 1 || a->span <= 0 || a->span % kQ) return -1;
  if (a->seg.count <= 0) return 0;
  if (static_cast<int64_t>(a->span) * a->parts < a->seg.max_len || a->seg.count > 65535 || a->parts > 65535) return -1;
  if (a->parts > 1 && (a->part_state == nullptr || a->part_decay == nullptr)) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a->n_state <= 64) return launch_ssd<64>(a, st);
  if (a->n_state <= 128) return launch_ssd<128>(a, st);
  if (a->n_state <= 256) return launch_ssd<256>(a, st);
  return -1;
}

extern "C" int64_t nx_delta_scratch_bytes(int heads, int segments, int max_len) {
  return static_cast<int64_t>(segments) * ((max_len + kQ - 1) / kQ) * heads * kDeltaUnit * 2;
}

extern "C" int nx_delta_chunk(const NxDeltaArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->dtype != NX_BF16 || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads) return -1;
  if (a->dim <= 0 || a->vdim <= 0) return -1;
  if (a->seg.count <= 0) return 0;
  if (a->scratch == nullptr || a->seg.count > 65535 || a->heads > 65535) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a->dim <= 64) return launch_delta<64>(a, st);
  if (a->dim <= 128) return launch_delta<128>(a, st);
  if (a->dim <= 256) return launch_delta<256>(a, st);
  return -1;
}
