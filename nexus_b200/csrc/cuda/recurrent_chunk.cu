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
#include "recurrent_common.cuh"

#include <algorithm>

namespace {
using namespace nx;

constexpr int kCols = 64;              // value columns per block (state-space)

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
// state-space duality.  grid (heads * column tiles, parts, segments), 8 warps.  Warp w owns 16 token rows of
// the chunk's outputs and NP / 4 rows of the state (w mod 4), 32 value columns of both (w / 4).
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
__global__ void __launch_bounds__(256, NP <= 128 ? 2 : 1) ssd_chunk_kernel(const NxSsdArgs a, int col_tiles) {
  using L = SsdSmem<NP>;
  constexpr int LN = L::LN, LP = L::LP, MT = NP / 64;    // MT: 16-row tiles of the state per warp
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16 *sB = sm + L::kB, *sC = sm + L::kC, *sX = sm + L::kX, *sXh = sm + L::kXh, *sXl = sm + L::kXl,
                *sSh = sm + L::kSh, *sSl = sm + L::kSl;
  __shared__ float s_c[kQ], s_dt[kQ], s_w[kQ];           // cumulative log2 decay, step size, weight in the new state
  const int h = blockIdx.x / col_tiles, p0 = (blockIdx.x % col_tiles) * kCols, part = blockIdx.y, sg = blockIdx.z;
  const int len = a.seg.len[sg], t_begin = part * a.span, t_end = min(len, t_begin + a.span);
  if (t_begin >= len || (kLocal && t_end == len)) return;   // the last span's contribution is never needed
  const int N = a.n_state, P = a.vdim, cols = min(kCols, P - p0), inner = a.heads * P, g = h / (a.heads / a.groups);
  const int warp = (threadIdx.x >> 5) & 3, cb = (threadIdx.x >> 7) * 32, lane = threadIdx.x & 31, qr = lane >> 2, qc = (lane & 3) * 2;
  const int64_t row0 = a.seg.row0[sg];
  const __nv_bfloat16* xbc = static_cast<const __nv_bfloat16*>(a.xbc) + row0 * a.ld_xbc;
  const __nv_bfloat16* dtp = static_cast<const __nv_bfloat16*>(a.dt) + row0 * a.ld_dt + h;
  const bool aligned = (a.ld_xbc & 7) == 0 && (inner & 7) == 0 && (reinterpret_cast<uintptr_t>(a.xbc) & 15) == 0;
  const bool vec_n = aligned && (N & 7) == 0, vec_p = aligned && (P & 7) == 0;
  const float rate = -expf(a.a_log[h]) * kLog2e, dtb = a.dt_bias[h], skip = a.d_skip[h];
  const int64_t plane = static_cast<int64_t>(N) * P;
  float* pool = a.state + (static_cast<int64_t>(a.seg.seq[sg]) * a.heads + h) * plane;
  float* part_state = a.parts > 1 ? a.part_state + ((static_cast<int64_t>(sg) * a.parts + part) * a.heads + h) * plane : nullptr;
  float S[MT][4][4];
  {
    const float* src = kLocal ? nullptr : a.parts > 1 ? part_state : (a.seg.pos[sg] == 0 ? nullptr : pool);
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = (warp * MT + m) * 16 + (e >> 1) * 8 + qr, c = cb + n * 8 + qc + (e & 1);
          S[m][n][e] = (src != nullptr && r < N && c < cols) ? src[static_cast<int64_t>(r) * P + p0 + c] : 0.0f;
        }
  }
  float total = 0.0f;                                    // log2 decay of the whole span
  auto load_cx = [&](int t0) {
    const __nv_bfloat16* src = xbc + t0 * a.ld_xbc;
    const int rows = min(kQ, t_end - t0);
    if (!kLocal) load_tile<NP>(sC, src + inner + (a.groups + g) * N, a.ld_xbc, rows, N, vec_n);
    load_tile<kCols>(sX, src + h * P + p0, a.ld_xbc, rows, cols, vec_p);
  };
  auto load_b = [&](int t0) {
    load_tile<NP>(sB, xbc + t0 * a.ld_xbc + inner + g * N, a.ld_xbc, min(kQ, t_end - t0), N, vec_n);
  };
  float raw[2];                                          // first warp: raw step sizes of the next chunk
  auto fetch_dt = [&](int t0) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = t0 + lane + 32 * i;
      raw[i] = t < t_end ? __bfloat162float(dtp[t * a.ld_dt]) : -INFINITY;      // softplus(-inf) = 0: no step
    }
  };
  auto scan_dt = [&] {
    float d[2], c[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      d[i] = raw[i] == -INFINITY ? 0.0f : softplus_exact(raw[i] + dtb);
      c[i] = rate * d[i];
    }
    scan64(c[0], c[1]);
    const float c_last = __shfl_sync(0xffffffffu, c[1], 31);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      s_dt[lane + 32 * i] = d[i];
      s_c[lane + 32 * i] = c[i];
      s_w[lane + 32 * i] = ex2_approx(c_last - c[i]) * d[i];
    }
  };
  load_cx(t_begin);
  load_b(t_begin);
  cp_async_commit();
  if (threadIdx.x < 32) {
    fetch_dt(t_begin);
    scan_dt();
    fetch_dt(t_begin + kQ);
  }
  for (int t0 = t_begin; t0 < t_end; t0 += kQ) {
    const int rows = min(kQ, t_end - t0);
    const bool more = t0 + kQ < t_end;
    if (!kLocal) {
#pragma unroll
      for (int m = 0; m < MT; ++m) store_split<4, LP>(sSh + cb, sSl + cb, (warp * MT + m) * 16, S[m]);
    }
    cp_async_wait<0>();
    __syncthreads();
    const float c_end = s_c[kQ - 1];
    // x weighted for the state update
    for (int i = threadIdx.x; i < kQ * (kCols / 2); i += 256) {
      const int t = i / (kCols / 2), o = t * LP + (i % (kCols / 2)) * 2;
      const float w = s_w[t];
      const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(sX + o);
      uint32_t hi, lo;
      bf16_split(__low2float(x) * w, __high2float(x) * w, hi, lo);
      *reinterpret_cast<uint32_t*>(sXh + o) = hi;
      *reinterpret_cast<uint32_t*>(sXl + o) = lo;
    }
    if (!kLocal) {
      const float ci[2] = {s_c[warp * 16 + qr], s_c[warp * 16 + 8 + qr]};
      float y[4][4];
      zero(y);
#pragma unroll
      for (int kk = 0; kk < NP / 16; ++kk) {             // C S
        uint32_t ca[4];
        ldmatrix_x4(ca, addr_a<LN>(sC, warp * 16, kk * 16));
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, addr_b_t<LP>(sSh, kk * 16, cb + n * 16));
          mma_bf16(y[2 * n], ca, b[0], b[1]);
          mma_bf16(y[2 * n + 1], ca, b[2], b[3]);
          ldmatrix_x4_trans(b, addr_b_t<LP>(sSl, kk * 16, cb + n * 16));
          mma_bf16(y[2 * n], ca, b[0], b[1]);
          mma_bf16(y[2 * n + 1], ca, b[2], b[3]);
        }
      }
      const float e0 = ex2_approx(ci[0]), e1 = ex2_approx(ci[1]);
#pragma unroll
      for (int n = 0; n < 4; ++n) {
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
            gm[n][e] = s <= t ? gm[n][e] * ex2_approx(ci[e >> 1] - s_c[s]) * s_dt[s] : 0.0f;
          }
        uint32_t mh[4], ml[4];
        bf16_split(gm[0][0], gm[0][1], mh[0], ml[0]);
        bf16_split(gm[0][2], gm[0][3], mh[1], ml[1]);
        bf16_split(gm[1][0], gm[1][1], mh[2], ml[2]);
        bf16_split(gm[1][2], gm[1][3], mh[3], ml[3]);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, addr_b_t<LP>(sX, j * 16, cb + n * 16));
          mma_bf16(y[2 * n], mh, b[0], b[1]);
          mma_bf16(y[2 * n + 1], mh, b[2], b[3]);
          mma_bf16(y[2 * n], ml, b[0], b[1]);
          mma_bf16(y[2 * n + 1], ml, b[2], b[3]);
        }
      }
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.y) + (row0 + t0) * a.ldy + static_cast<int64_t>(h) * P + p0;
      const bool pair = ((a.ldy | P) & 1) == 0;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = warp * 16 + i * 8 + qr;
        if (t >= rows) continue;
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          const int c = cb + n * 8 + qc;
          const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(sX + t * LP + c);
          const float v0 = y[n][2 * i] + skip * __low2float(x), v1 = y[n][2 * i + 1] + skip * __high2float(x);
          if (pair) {
            if (c < cols) *reinterpret_cast<uint32_t*>(out + t * a.ldy + c) = bf16_pair(v0, v1);
          } else {
            if (c < cols) out[t * a.ldy + c] = __float2bfloat16_rn(v0);
            if (c + 1 < cols) out[t * a.ldy + c + 1] = __float2bfloat16_rn(v1);
          }
        }
      }
    }
    __syncthreads();                                     // weighted x complete; C, x and the step sizes are free again
    if (more) {
      load_cx(t0 + kQ);
      if (threadIdx.x < 32) {
        scan_dt();
        fetch_dt(t0 + 2 * kQ);
      }
    }
    const float dec = ex2_approx(c_end);
    total += c_end;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][n][e] *= dec;
#pragma unroll
    for (int kk = 0; kk < kQ / 16; ++kk) {
      uint32_t ba[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldmatrix_x4_trans(ba[m], addr_a_t<LN>(sB, kk * 16, (warp * MT + m) * 16));
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bh, addr_b_t<LP>(sXh, kk * 16, cb + n * 16));
        ldmatrix_x4_trans(bl, addr_b_t<LP>(sXl, kk * 16, cb + n * 16));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16(S[m][2 * n], ba[m], bh[0], bh[1]);
          mma_bf16(S[m][2 * n + 1], ba[m], bh[2], bh[3]);
          mma_bf16(S[m][2 * n], ba[m], bl[0], bl[1]);
          mma_bf16(S[m][2 * n + 1], ba[m], bl[2], bl[3]);
        }
      }
    }
    __syncthreads();                                     // B is free
    if (more) {
      load_b(t0 + kQ);
      cp_async_commit();
    }
  }
  float* dst = kLocal ? part_state : (t_end == len ? pool : nullptr);
  if (dst != nullptr) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = (warp * MT + m) * 16 + (e >> 1) * 8 + qr, c = cb + n * 8 + qc + (e & 1);
          if (r < N && c < cols) dst[static_cast<int64_t>(r) * P + p0 + c] = S[m][n][e];
        }
    if (kLocal && threadIdx.x == 0 && p0 == 0)
      a.part_decay[(static_cast<int64_t>(sg) * a.parts + part) * a.heads + h] = ex2_approx(total);
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
    ssd_chunk_kernel<NP, true><<<grid, 256, kBytes, st>>>(*a, col_tiles);
    const int plane = a->n_state * a->vdim;
    ssd_span_scan_kernel<<<dim3(a->heads, a->seg.count, (plane + 255) / 256), 256, 0, st>>>(*a);
  }
  ssd_chunk_kernel<NP, false><<<grid, 256, kBytes, st>>>(*a, col_tiles);
  return launch_status();
}

// ------------------------------------------------------------------------------------------------
// delta rule, first kernel: everything of a chunk that does not depend on the state.
// grid (chunks, heads, segments), 4 warps.  Scratch per (segment, chunk, head): T hi | T lo | P hi | P lo, each 64 x 64 BF16
// in the order of the A fragments that read them - [row tile][16-column block][lane][8], blocks past the diagonal unused -
// then FP32 [4][64]: cumulative log2 decay, 1 / |k|, dim^-1/2 / |q|, beta.
// ------------------------------------------------------------------------------------------------
constexpr int64_t kDeltaTile = kQ * kQ;
constexpr int64_t kDeltaUnit = 4 * kDeltaTile + 4 * kQ * 2;   // in BF16 elements

__device__ __forceinline__ uint4* fragment(__nv_bfloat16* tile, int row_tile, int block) {
  return reinterpret_cast<uint4*>(tile) + (row_tile * (kQ / 16) + block) * 32 + (threadIdx.x & 31);
}
__device__ __forceinline__ void store_fragment(__nv_bfloat16* hi, __nv_bfloat16* lo, int row_tile, int block, const float (&v)[2][4]) {
  uint4 h, l;                          // v: two 16 x 8 accumulator tiles side by side
  bf16_split(v[0][0], v[0][1], h.x, l.x);
  bf16_split(v[0][2], v[0][3], h.y, l.y);
  bf16_split(v[1][0], v[1][1], h.z, l.z);
  bf16_split(v[1][2], v[1][3], h.w, l.w);
  *fragment(hi, row_tile, block) = h;
  *fragment(lo, row_tile, block) = l;
}

// bytes of the first region of the kernel's shared memory: q and k, later the inverse and its scratch
template <int DP>
constexpr int prep_front() {
  constexpr int qk = 2 * kQ * (DP + 8) * 2, inv = (kQ * (kQ + 4) + 4 * 16 * 17) * 4;
  return qk > inv ? qk : inv;
}

// acc[r] += sum_k a[r][k] b[k], 8 rows of `a` (pitch LA, 16-byte aligned) and one column of `b` (pitch LB), n a multiple of 4
template <int LA, int LB = LA>
__device__ __forceinline__ void block_product(float (&acc)[8], const float* a, const float* b, int n) {
  for (int k = 0; k < n; k += 4) {
    float bv[4];
#pragma unroll
    for (int q = 0; q < 4; ++q) bv[q] = b[(k + q) * LB];
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      const float4 av = *reinterpret_cast<const float4*>(a + r * LA + k);
      acc[r] += av.x * bv[0] + av.y * bv[1] + av.z * bv[2] + av.w * bv[3];
    }
  }
}

template <int DP>
__global__ void __launch_bounds__(128) delta_prep_kernel(const NxDeltaArgs a, int chunks) {
  constexpr int LD = DP + 8, LA = kQ + 4;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16 *sK = sm, *sQ = sm + kQ * LD;
  float* sT = reinterpret_cast<float*>(sm);                   // [64][LA], then [4][16][17]: over q and k, once these are consumed
  float* sW = sT + kQ * LA;
  float* sA = sT + prep_front<DP>() / 4;                      // [64][LA]
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
  for (int j = 0; j <= warp; ++j) {
    float kk[2][4], qk[2][4];
    zero(kk);
    zero(qk);
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
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = e >> 1, t = warp * 16 + i * 8 + qr, s = j * 16 + n * 8 + qc + (e & 1);
        const float w = s <= t ? ex2_approx(bt[i] - s_b[s]) * s_rk[s] : 0.0f;
        qk[n][e] *= w * rqt[i];
        sA[t * LA + s] = s < t ? kk[n][e] * w * rkt[i] * bet[i] : 0.0f;
      }
    store_fragment(Ph, Pl, warp, j, qk);
  }
  __syncthreads();
  // T = (I + A)^-1 by 16 x 16 blocks, FP32.  Diagonal blocks: one thread per column, forward substitution in registers.
  if (threadIdx.x < kQ) {
    const int blk = threadIdx.x / 16 * 16, c = threadIdx.x % 16;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float v = i == c ? 1.0f : 0.0f;
#pragma unroll
      for (int j = 0; j < i; ++j) v -= sA[(blk + i) * LA + blk + j] * x[j];
      x[i] = v;
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) sT[(blk + i) * LA + blk + c] = x[i];
  }
  // Below the diagonal: T_ij = -T_ii sum_{j <= k < i} A_ik T_kj, one block diagonal after the other, a warp per block.  A lane
  // has one column and 8 rows.
  for (int d = 1; d < kQ / 16; ++d) {
    __syncthreads();
    const int i = warp + d, j = warp;
    if (i < kQ / 16) {
      const int c = lane & 15, r0 = (lane >> 4) * 8;
      float acc[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
      block_product<LA>(acc, sA + (i * 16 + r0) * LA + j * 16, sT + j * 16 * LA + j * 16 + c, 16 * d);
      float* w = sW + warp * 16 * 17;
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        w[(r0 + r) * 17 + c] = acc[r];
        acc[r] = 0.0f;
      }
      __syncwarp();
      block_product<LA, 17>(acc, sT + (i * 16 + r0) * LA + i * 16, w + c, 16);
#pragma unroll
      for (int r = 0; r < 8; ++r) sT[(i * 16 + r0 + r) * LA + j * 16 + c] = -acc[r];
    }
  }
  __syncthreads();
  for (int j = 0; j <= warp; ++j) {
    float v[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) v[n][e] = sT[(warp * 16 + (e >> 1) * 8 + qr) * LA + j * 16 + n * 8 + qc + (e & 1)];
    store_fragment(Th, Tl, warp, j, v);
  }
  if (threadIdx.x < kQ) {
    const int c = threadIdx.x;
    float* sc = reinterpret_cast<float*>(unit + 4 * kDeltaTile);
    sc[c] = s_b[c];
    sc[kQ + c] = s_rk[c];
    sc[2 * kQ + c] = s_rq[c];
    sc[3 * kQ + c] = s_beta[c];
  }
}

// ------------------------------------------------------------------------------------------------
// delta rule, second kernel: the chunks of a segment in order.  grid (heads * column tiles, segments),
// 8 warps: warp w owns 16 token rows of U and the outputs and DP / 4 rows of the state (w mod 4), half
// of the block's COLS value columns of both (w / 4).
// ------------------------------------------------------------------------------------------------
template <int DP, int COLS>
struct DeltaSmem {
  static constexpr int LD = DP + 8, LV = COLS + 8;
  static constexpr int kK = 0, kQq = kK + kQ * LD, kRh = kQq + kQ * LD, kRl = kRh + kQ * LV, kUh = kRl + kQ * LV,
                       kUl = kUh + kQ * LV, kSh = kUl + kQ * LV, kSl = kSh + DP * LV, kEnd = kSl + DP * LV;
  static constexpr int kBytes = kEnd * 2;
};

// d += (ah + al) (bh + bl) up to the product of the two remainders, over the blocks 0 .. row_tile of a lower-triangular tile
// pair in fragment order; d covers 8 NT columns
template <int LV, int NT>
__device__ __forceinline__ void mma_triangle(float (&d)[NT][4], const uint4 (&ah)[kQ / 16], const uint4 (&al)[kQ / 16],
                                             const __nv_bfloat16* bh, const __nv_bfloat16* bl, int row_tile, int col) {
#pragma unroll
  for (int kk = 0; kk < kQ / 16; ++kk) {
    if (kk > row_tile) break;
    const uint32_t fh[4] = {ah[kk].x, ah[kk].y, ah[kk].z, ah[kk].w}, fl[4] = {al[kk].x, al[kk].y, al[kk].z, al[kk].w};
#pragma unroll
    for (int n = 0; n < NT / 2; ++n) {
      uint32_t gh[4], gl[4];
      ldmatrix_x4_trans(gh, addr_b_t<LV>(bh, kk * 16, col + n * 16));
      ldmatrix_x4_trans(gl, addr_b_t<LV>(bl, kk * 16, col + n * 16));
      mma_bf16(d[2 * n], fh, gh[0], gh[1]);
      mma_bf16(d[2 * n + 1], fh, gh[2], gh[3]);
      mma_bf16(d[2 * n], fh, gl[0], gl[1]);
      mma_bf16(d[2 * n + 1], fh, gl[2], gl[3]);
      mma_bf16(d[2 * n], fl, gh[0], gh[1]);
      mma_bf16(d[2 * n + 1], fl, gh[2], gh[3]);
    }
  }
}
__device__ __forceinline__ void load_fragments(uint4 (&hi)[kQ / 16], uint4 (&lo)[kQ / 16], const __nv_bfloat16* tile, int row_tile) {
#pragma unroll
  for (int kk = 0; kk < kQ / 16; ++kk) {
    if (kk > row_tile) break;
    hi[kk] = *fragment(const_cast<__nv_bfloat16*>(tile), row_tile, kk);
    lo[kk] = *fragment(const_cast<__nv_bfloat16*>(tile) + kDeltaTile, row_tile, kk);
  }
}

template <int DP, int COLS>
__global__ void __launch_bounds__(256, DP <= 128 ? 2 : 1) delta_chunk_kernel(const NxDeltaArgs a, int chunks, int col_tiles) {
  using L = DeltaSmem<DP, COLS>;
  constexpr int LD = L::LD, LV = L::LV, MT = DP / 64, NT = COLS / 16;    // NT: 8-column tiles per warp
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16 *sK = sm + L::kK, *sQ = sm + L::kQq, *sRh = sm + L::kRh, *sRl = sm + L::kRl, *sUh = sm + L::kUh, *sUl = sm + L::kUl,
                *sSh = sm + L::kSh, *sSl = sm + L::kSl;
  __nv_bfloat16* sV = sUh;             // v is consumed before U is written
  __shared__ __align__(16) float s_sc[4 * kQ];           // cumulative log2 decay | 1/|k| | scaled 1/|q| | beta
  const int h = blockIdx.x / col_tiles, v0 = (blockIdx.x % col_tiles) * COLS, sg = blockIdx.y;
  const int len = a.seg.len[sg];
  if (len <= 0) return;
  const int D = a.dim, Dv = a.vdim, cols = min(COLS, Dv - v0), hk = h / (a.heads / a.kv_heads), kcols = a.kv_heads * D;
  const int warp = (threadIdx.x >> 5) & 3, cb = (threadIdx.x >> 7) * (COLS / 2), lane = threadIdx.x & 31, qr = lane >> 2, qc = (lane & 3) * 2;
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
        const int r = (warp * MT + m) * 16 + (e >> 1) * 8 + qr, c = cb + n * 8 + qc + (e & 1);
        S[m][n][e] = (!fresh && r < D && c < cols) ? pool[static_cast<int64_t>(r) * Dv + v0 + c] : 0.0f;
      }
  const __nv_bfloat16* qsrc = static_cast<const __nv_bfloat16*>(a.qkv) + row0 * a.ld_qkv + hk * D;
  load_tile<DP>(sQ, qsrc, a.ld_qkv, min(kQ, len), D, vec_d);
  for (int ch = 0; ch * kQ < len; ++ch) {
    const int t0 = ch * kQ, rows = min(kQ, len - t0);
    const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(a.qkv) + (row0 + t0) * a.ld_qkv;
    const __nv_bfloat16* unit = static_cast<const __nv_bfloat16*>(a.scratch) +
                                ((static_cast<int64_t>(sg) * chunks + ch) * a.heads + h) * kDeltaUnit;
    load_tile<DP>(sK, src + kcols + hk * D, a.ld_qkv, rows, D, vec_d);
    load_tile<COLS>(sV, src + 2 * kcols + h * Dv + v0, a.ld_qkv, rows, cols, vec_v);
    if (threadIdx.x < kQ) cp_async16(s_sc + threadIdx.x * 4, reinterpret_cast<const float*>(unit + 4 * kDeltaTile) + threadIdx.x * 4);
    cp_async_commit();
    uint4 fh[kQ / 16], fl[kQ / 16];                      // rows of T, later of P
    load_fragments(fh, fl, unit, warp);
#pragma unroll
    for (int m = 0; m < MT; ++m) store_split<NT, LV>(sSh + cb, sSl + cb, (warp * MT + m) * 16, S[m]);
    cp_async_wait<0>();
    __syncthreads();
    const float b_end = s_sc[kQ - 1];
    float o[NT][4], u[NT][4];
    zero(o);
    {
      float ks[NT][4];
      zero(ks);
#pragma unroll
      for (int d = 0; d < DP / 16; ++d) {
        uint32_t ka[4], qa[4];
        ldmatrix_x4(ka, addr_a<LD>(sK, warp * 16, d * 16));
        ldmatrix_x4(qa, addr_a<LD>(sQ, warp * 16, d * 16));
#pragma unroll
        for (int n = 0; n < NT / 2; ++n) {
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(bh, addr_b_t<LV>(sSh, d * 16, cb + n * 16));
          ldmatrix_x4_trans(bl, addr_b_t<LV>(sSl, d * 16, cb + n * 16));
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
      for (int i = 0; i < 2; ++i) {
        const int t = warp * 16 + i * 8 + qr;
        const float eb = ex2_approx(s_sc[t]), fk = eb * s_sc[kQ + t], fq = eb * s_sc[2 * kQ + t], beta = s_sc[3 * kQ + t];
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(sV + t * LV + cb + n * 8 + qc);
          ks[n][2 * i] = beta * (__low2float(v) - fk * ks[n][2 * i]);
          ks[n][2 * i + 1] = beta * (__high2float(v) - fk * ks[n][2 * i + 1]);
          o[n][2 * i] *= fq;
          o[n][2 * i + 1] *= fq;
        }
      }
      store_split<NT, LV>(sRh + cb, sRl + cb, warp * 16, ks);
    }
    __syncthreads();
    zero(u);
    mma_triangle<LV, NT>(u, fh, fl, sRh, sRl, warp, cb);
    load_fragments(fh, fl, unit + 2 * kDeltaTile, warp);
    store_split<NT, LV>(sUh + cb, sUl + cb, warp * 16, u);
    __syncthreads();                                     // U complete, R no longer read: it takes the weighted U
    if (t0 + kQ < len) load_tile<DP>(sQ, qsrc + (t0 + kQ) * a.ld_qkv, a.ld_qkv, min(kQ, len - t0 - kQ), D, vec_d);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = warp * 16 + i * 8 + qr;
      const float w = ex2_approx(b_end - s_sc[t]) * s_sc[kQ + t];
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        u[n][2 * i] *= w;
        u[n][2 * i + 1] *= w;
      }
    }
    store_split<NT, LV>(sRh + cb, sRl + cb, warp * 16, u);
    mma_triangle<LV, NT>(o, fh, fl, sUh, sUl, warp, cb);
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.o) + (row0 + t0) * a.ldo + static_cast<int64_t>(h) * Dv + v0;
    const bool pair = ((a.ldo | Dv) & 1) == 0;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = warp * 16 + i * 8 + qr;
      if (t >= rows) continue;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int c = cb + n * 8 + qc;
        if (pair) {
          if (c < cols) *reinterpret_cast<uint32_t*>(out + t * a.ldo + c) = bf16_pair(o[n][2 * i], o[n][2 * i + 1]);
        } else {
          if (c < cols) out[t * a.ldo + c] = __float2bfloat16_rn(o[n][2 * i]);
          if (c + 1 < cols) out[t * a.ldo + c + 1] = __float2bfloat16_rn(o[n][2 * i + 1]);
        }
      }
    }
    __syncthreads();
    const float dec = ex2_approx(b_end);
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
        ldmatrix_x4_trans(bh, addr_b_t<LV>(sRh, kk * 16, cb + n * 16));
        ldmatrix_x4_trans(bl, addr_b_t<LV>(sRl, kk * 16, cb + n * 16));
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
        const int r = (warp * MT + m) * 16 + (e >> 1) * 8 + qr, c = cb + n * 8 + qc + (e & 1);
        if (r < D && c < cols) pool[static_cast<int64_t>(r) * Dv + v0 + c] = S[m][n][e];
      }
}

template <int DP, int COLS>
int launch_delta_chunks(const NxDeltaArgs* a, int chunks, cudaStream_t st) {
  constexpr int kBytes = DeltaSmem<DP, COLS>::kBytes;
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(delta_chunk_kernel<DP, COLS>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes) != cudaSuccess) return -2;
    once = true;
  }
  const int col_tiles = (a->vdim + COLS - 1) / COLS;
  delta_chunk_kernel<DP, COLS><<<dim3(a->heads * col_tiles, a->seg.count), 256, kBytes, st>>>(*a, chunks, col_tiles);
  return launch_status();
}

template <int DP>
int launch_delta(const NxDeltaArgs* a, cudaStream_t st) {
  constexpr int kPrep = prep_front<DP>() + kQ * (kQ + 4) * 4;
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(delta_prep_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPrep) != cudaSuccess) return -2;
    once = true;
  }
  const int chunks = (a->seg.max_len + kQ - 1) / kQ;
  delta_prep_kernel<DP><<<dim3(chunks, a->heads, a->seg.count), 128, kPrep, st>>>(*a, chunks);
  // the chunks of a segment are a chain: while the blocks do not fill the GPU, narrower column tiles shorten every link
  const int wide = a->heads * ((a->vdim + 63) / 64) * a->seg.count;
  return wide < kNumSmsB200 && a->vdim > 32 ? launch_delta_chunks<DP, 32>(a, chunks, st) : launch_delta_chunks<DP, 64>(a, chunks, st);
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
