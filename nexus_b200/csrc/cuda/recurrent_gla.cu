// Chunked tensor-core form of gated linear attention (see nx_api_mixers.h) for long segments with BF16 activations: a decay per
// key channel and token.  A chunk is 64 tokens in four sub-blocks of 16; a block carries the FP32 state of one head (one tile of
// value columns of it) through the chunks of its segment in registers, as the accumulators of the products that update it.
//
// Per channel, c_t = a_1 + .. + a_t is the log2 decay since the start of the token's sub-block, R_j the total of sub-block j.
// The convert step forms, once per chunk,
//   q^_t = q_scale q_t 2^{c_t}          (from the start of t's sub-block; the exponent is <= 0)
//   k^_s = k_s 2^{R_j - c_s}            (to the end of s's sub-block; the exponent is <= 0)
// and everything else needs only factors that are the same for all tokens of a sub-block:
//   y_t  = sum_d q^_t 2^{R_0 + .. + R_{i-1}} S  +  sum_{s <= t} (sum_d q^_t F_ij k^_s) v_s,   t in sub-block i, s in j
//          F_ij = 2^{R_{j+1} + .. + R_{i-1}} for j < i,   F_ii = 2^{-R_i}
//   S'   : S = 2^{R_j} S + k^_j^T v_j for j = 0 .. 3
// Only F_ii grows with the decay.  Where a sub-block decays by more than 2^60 its own 16 x 16 products are formed pair by pair
// from the exponents' differences instead, so any decay is exact.
//
// Precision: v is BF16 and enters as it is; q^, k^, S and the token-by-token products are FP32 values split into BF16 pairs
// (value and rounding remainder), which keeps 16 bits of mantissa.
#include "recurrent_common.cuh"

#include <algorithm>

namespace {
using namespace nx;

constexpr int kCols = 64;              // value columns per block
constexpr int kSub = 16;               // tokens per sub-block
constexpr float kSafe = -60.0f;        // smallest R whose inverse is used

template <int NP>
struct Smem {
  static constexpr int LN = NP + 8, LP = kCols + 8;
  static constexpr int kQh = 0, kQl = kQh + kQ * LN, kKh = kQl + kQ * LN, kKl = kKh + kQ * LN, kV = kKl + kQ * LN,
                       kSh = kV + kQ * LP, kSl = kSh + NP * LP, kEnd = kSl + NP * LP;
  static constexpr int kBytes = kEnd * 2 + 4 * NP * 4;
};

// a fragment pair (value, remainder) times one factor per column: f = columns qc, qc + 1, qc + 8, qc + 9
__device__ __forceinline__ void scale_pair(uint32_t (&h)[4], uint32_t (&l)[4], const float (&f)[4]) {
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(&h[r]), y = *reinterpret_cast<const __nv_bfloat162*>(&l[r]);
    const int i = (r >> 1) * 2;
    bf16_split((__low2float(x) + __low2float(y)) * f[i], (__high2float(x) + __high2float(y)) * f[i + 1], h[r], l[r]);
  }
}

// grid (heads * column tiles, parts, segments), 8 warps.  Warp w owns sub-block w mod 4 of the outputs and NP / 4 rows of the
// state, 32 value columns of both (w / 4).  kLocal: only the span's own contribution to the state, from zero, and its decay (for
// spans that run at the same time); otherwise outputs, from the span's true start state.
template <int NP, bool kLocal>
__global__ void __launch_bounds__(256, NP <= 64 ? 2 : 1) gla_chunk_kernel(const NxGlaArgs a, int col_tiles) {
  using L = Smem<NP>;
  constexpr int LN = L::LN, LP = L::LP, MT = NP / 64, ITEMS = NP / 64;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16 *sQh = sm + L::kQh, *sQl = sm + L::kQl, *sKh = sm + L::kKh, *sKl = sm + L::kKl, *sV = sm + L::kV, *sSh = sm + L::kSh,
                *sSl = sm + L::kSl;
  float* sR = reinterpret_cast<float*>(sm + L::kEnd);    // [4][NP]: log2 decay of every sub-block
  __shared__ int s_far[2][4];                            // sub-blocks whose decay is not inverted, by chunk parity
  const int h = blockIdx.x / col_tiles, p0 = (blockIdx.x % col_tiles) * kCols, part = blockIdx.y, sg = blockIdx.z;
  const int len = a.seg.len[sg], t_begin = part * a.span, t_end = min(len, t_begin + a.span);
  if (t_begin >= len || (kLocal && t_end == len)) return;   // the last span's contribution is never needed
  const int D = a.dim, P = a.vdim, cols = min(kCols, P - p0);
  const int warp = (threadIdx.x >> 5) & 3, cb = (threadIdx.x >> 7) * 32, lane = threadIdx.x & 31, qr = lane >> 2, qc = (lane & 3) * 2;
  const int64_t row0 = a.seg.row0[sg];
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + row0 * a.ld + static_cast<int64_t>(h) * D;
  const __nv_bfloat16* k = static_cast<const __nv_bfloat16*>(a.k) + row0 * a.ld + static_cast<int64_t>(h) * D;
  const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(a.v) + row0 * a.ld + static_cast<int64_t>(h) * P + p0;
  const float* dec = a.decay + row0 * a.ld_decay + static_cast<int64_t>(h) * D;
  const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec_d = (a.ld & 7) == 0 && (D & 7) == 0 && al(a.q) && al(a.k), vec_p = (a.ld & 7) == 0 && (P & 7) == 0 && al(a.v);
  const int64_t plane = static_cast<int64_t>(D) * P;
  float* pool = a.state + (static_cast<int64_t>(a.seg.seq[sg]) * a.heads + h) * plane;
  const int64_t unit = (static_cast<int64_t>(sg) * a.parts + part) * a.heads + h;
  float* part_state = a.parts > 1 ? a.part_state + unit * plane : nullptr;
  float S[MT][4][4], total[MT][2];
  {
    const float* src = kLocal ? nullptr : a.parts > 1 ? part_state : (a.seg.pos[sg] == 0 ? nullptr : pool);
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      total[m][0] = total[m][1] = 0.0f;
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = (warp * MT + m) * 16 + (e >> 1) * 8 + qr, c = cb + n * 8 + qc + (e & 1);
          S[m][n][e] = (src != nullptr && r < D && c < cols) ? src[static_cast<int64_t>(r) * P + p0 + c] : 0.0f;
        }
    }
  }
  auto load_q = [&](int t0) { load_tile<NP>(sQh, q + t0 * a.ld, a.ld, min(kQ, t_end - t0), D, vec_d); };
  auto load_kv = [&](int t0) {
    load_tile<NP>(sKh, k + t0 * a.ld, a.ld, min(kQ, t_end - t0), D, vec_d);
    load_tile<kCols>(sV, v + t0 * a.ld, a.ld, min(kQ, t_end - t0), cols, vec_p);
  };
  float raw[ITEMS][kSub];                                // log2 decays of the chunk to convert next: one channel, one sub-block
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int item = threadIdx.x + i * 256, d = item % NP, t = t0 + item / NP * kSub;
#pragma unroll
      for (int u = 0; u < kSub; ++u) raw[i][u] = d < D && t + u < t_end ? dec[static_cast<int64_t>(t + u) * a.ld_decay + d] : 0.0f;
    }
  };
  if (!kLocal) load_q(t_begin);
  load_kv(t_begin);
  cp_async_commit();
  fetch(t_begin);
  if (threadIdx.x < 8) s_far[threadIdx.x >> 2][threadIdx.x & 3] = 0;
  int par = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += kQ, par ^= 1) {
    const int rows = min(kQ, t_end - t0);
    const bool more = t0 + kQ < t_end;
    if (!kLocal) {
#pragma unroll
      for (int m = 0; m < MT; ++m) store_split<4, LP>(sSh + cb, sSl + cb, (warp * MT + m) * 16, S[m]);
    }
    cp_async_wait<0>();
    __syncthreads();
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int item = threadIdx.x + i * 256, d = item % NP, j = item / NP;
#pragma unroll
      for (int u = 1; u < kSub; ++u) raw[i][u] += raw[i][u - 1];
      const float end = raw[i][kSub - 1];
      sR[j * NP + d] = end;
      if (end < kSafe) s_far[par][j] = 1;
#pragma unroll
      for (int u = 0; u < kSub; ++u) {
        const int o = (j * kSub + u) * LN + d;
        if (!kLocal) {
          const float x = __bfloat162float(sQh[o]) * (a.q_scale * ex2_approx(raw[i][u]));
          const __nv_bfloat16 hi = __float2bfloat16_rn(x);
          sQh[o] = hi;
          sQl[o] = __float2bfloat16_rn(x - __bfloat162float(hi));
        }
        const float x = __bfloat162float(sKh[o]) * ex2_approx(end - raw[i][u]);
        const __nv_bfloat16 hi = __float2bfloat16_rn(x);
        sKh[o] = hi;
        sKl[o] = __float2bfloat16_rn(x - __bfloat162float(hi));
      }
    }
    if (more) fetch(t0 + kQ);
    __syncthreads();
    if (threadIdx.x < 4) s_far[par ^ 1][threadIdx.x] = 0;
    if (!kLocal) {
      // 2^(sum of R over sub-blocks j0 .. j1 - 1), times -1 in the exponent where `inverse`, for the lane's four channels
      auto factors = [&](int kk, int j0, int j1, bool inverse, float (&f)[4]) {
        float2 s0 = make_float2(0.0f, 0.0f), s1 = s0;
        for (int j = j0; j < j1; ++j) {
          const float2 r0 = *reinterpret_cast<const float2*>(sR + j * NP + kk * 16 + qc);
          const float2 r1 = *reinterpret_cast<const float2*>(sR + j * NP + kk * 16 + 8 + qc);
          s0.x += r0.x;
          s0.y += r0.y;
          s1.x += r1.x;
          s1.y += r1.y;
        }
        const float sign = inverse ? -1.0f : 1.0f;
        f[0] = ex2_approx(sign * s0.x);
        f[1] = ex2_approx(sign * s0.y);
        f[2] = ex2_approx(sign * s1.x);
        f[3] = ex2_approx(sign * s1.y);
      };
      float y[4][4];
      zero(y);
#pragma unroll
      for (int kk = 0; kk < NP / 16; ++kk) {             // q S
        uint32_t qh[4], ql[4];
        ldmatrix_x4(qh, addr_a<LN>(sQh, warp * 16, kk * 16));
        ldmatrix_x4(ql, addr_a<LN>(sQl, warp * 16, kk * 16));
        if (warp > 0) {
          float f[4];
          factors(kk, 0, warp, false, f);
          scale_pair(qh, ql, f);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(bh, addr_b_t<LP>(sSh, kk * 16, cb + n * 16));
          ldmatrix_x4_trans(bl, addr_b_t<LP>(sSl, kk * 16, cb + n * 16));
          mma_bf16(y[2 * n], qh, bh[0], bh[1]);
          mma_bf16(y[2 * n + 1], qh, bh[2], bh[3]);
          mma_bf16(y[2 * n], qh, bl[0], bl[1]);
          mma_bf16(y[2 * n + 1], qh, bl[2], bl[3]);
          mma_bf16(y[2 * n], ql, bh[0], bh[1]);
          mma_bf16(y[2 * n + 1], ql, bh[2], bh[3]);
        }
      }
      for (int j = 0; j <= warp; ++j) {                  // 16 keys at a time, up to the diagonal
        float g[2][4];
        zero(g);
        if (j == warp && s_far[par][warp]) {
          // the decay between two tokens directly: lane t < 16 holds token t of the sub-block
          const int t = t0 + warp * kSub + (lane & 15);
          const bool in = t < t_end;
          for (int d = 0; d < D; ++d) {
            float c = in ? dec[static_cast<int64_t>(t) * a.ld_decay + d] : 0.0f;
            const float qv = in ? a.q_scale * __bfloat162float(q[t * a.ld + d]) : 0.0f;
            const float kv = in ? __bfloat162float(k[t * a.ld + d]) : 0.0f;
#pragma unroll
            for (int o = 1; o < 16; o <<= 1) {
              const float x = __shfl_up_sync(0xffffffffu, c, o, 16);
              if ((lane & 15) >= o) c += x;
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) {
              const int r = (e >> 1 & 1) * 8 + qr, s = (e >> 2) * 8 + qc + (e & 1);
              const float cr = __shfl_sync(0xffffffffu, c, r), cs = __shfl_sync(0xffffffffu, c, s);
              const float qq = __shfl_sync(0xffffffffu, qv, r), kq = __shfl_sync(0xffffffffu, kv, s);
              g[e >> 2][e & 3] += qq * kq * ex2_approx(fminf(cr - cs, 0.0f));
            }
          }
        } else {
#pragma unroll
          for (int kk = 0; kk < NP / 16; ++kk) {
            uint32_t qh[4], ql[4], bh[4], bl[4];
            ldmatrix_x4(qh, addr_a<LN>(sQh, warp * 16, kk * 16));
            ldmatrix_x4(ql, addr_a<LN>(sQl, warp * 16, kk * 16));
            ldmatrix_x4(bh, addr_b<LN>(sKh, j * 16, kk * 16));
            ldmatrix_x4(bl, addr_b<LN>(sKl, j * 16, kk * 16));
            if (j != warp - 1) {
              float f[4];
              if (j == warp) factors(kk, warp, warp + 1, true, f);
              else factors(kk, j + 1, warp, false, f);
              scale_pair(qh, ql, f);
            }
            mma_bf16(g[0], qh, bh[0], bh[1]);
            mma_bf16(g[1], qh, bh[2], bh[3]);
            mma_bf16(g[0], qh, bl[0], bl[1]);
            mma_bf16(g[1], qh, bl[2], bl[3]);
            mma_bf16(g[0], ql, bh[0], bh[1]);
            mma_bf16(g[1], ql, bh[2], bh[3]);
          }
        }
        if (j == warp) {
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e)
              if (n * 8 + qc + (e & 1) > (e >> 1) * 8 + qr) g[n][e] = 0.0f;
        }
        uint32_t mh[4], ml[4];
        bf16_split(g[0][0], g[0][1], mh[0], ml[0]);
        bf16_split(g[0][2], g[0][3], mh[1], ml[1]);
        bf16_split(g[1][0], g[1][1], mh[2], ml[2]);
        bf16_split(g[1][2], g[1][3], mh[3], ml[3]);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, addr_b_t<LP>(sV, j * 16, cb + n * 16));
          mma_bf16(y[2 * n], mh, b[0], b[1]);
          mma_bf16(y[2 * n + 1], mh, b[2], b[3]);
          mma_bf16(y[2 * n], ml, b[0], b[1]);
          mma_bf16(y[2 * n + 1], ml, b[2], b[3]);
        }
      }
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.o) + (row0 + t0) * a.ldo + static_cast<int64_t>(h) * P + p0;
      const bool pair = ((a.ldo | P) & 1) == 0 && (reinterpret_cast<uintptr_t>(a.o) & 3) == 0;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = warp * 16 + i * 8 + qr;
        if (t >= rows) continue;
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          const int c = cb + n * 8 + qc;
          if (pair) {
            if (c < cols) *reinterpret_cast<uint32_t*>(out + t * a.ldo + c) = bf16_pair(y[n][2 * i], y[n][2 * i + 1]);
          } else {
            if (c < cols) out[t * a.ldo + c] = __float2bfloat16_rn(y[n][2 * i]);
            if (c + 1 < cols) out[t * a.ldo + c + 1] = __float2bfloat16_rn(y[n][2 * i + 1]);
          }
        }
      }
      __syncthreads();                                   // q is free
      if (more) load_q(t0 + kQ);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      uint32_t kh[MT][4], kl[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const int r = (warp * MT + m) * 16;
        ldmatrix_x4_trans(kh[m], addr_a_t<LN>(sKh, j * 16, r));
        ldmatrix_x4_trans(kl[m], addr_a_t<LN>(sKl, j * 16, r));
        const float r0 = sR[j * NP + r + qr], r1 = sR[j * NP + r + 8 + qr];
        const float d0 = ex2_approx(r0), d1 = ex2_approx(r1);
        total[m][0] += r0;
        total[m][1] += r1;
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          S[m][n][0] *= d0;
          S[m][n][1] *= d0;
          S[m][n][2] *= d1;
          S[m][n][3] *= d1;
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        uint32_t b[4];
        ldmatrix_x4_trans(b, addr_b_t<LP>(sV, j * 16, cb + n * 16));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16(S[m][2 * n], kh[m], b[0], b[1]);
          mma_bf16(S[m][2 * n + 1], kh[m], b[2], b[3]);
          mma_bf16(S[m][2 * n], kl[m], b[0], b[1]);
          mma_bf16(S[m][2 * n + 1], kl[m], b[2], b[3]);
        }
      }
    }
    __syncthreads();                                     // k, v and the decays are free
    if (more) {
      load_kv(t0 + kQ);
      cp_async_commit();
    }
  }
  float* dst = kLocal ? part_state : (t_end == len ? pool : nullptr);
  if (dst == nullptr) return;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = (warp * MT + m) * 16 + (e >> 1) * 8 + qr, c = cb + n * 8 + qc + (e & 1);
        if (r < D && c < cols) dst[static_cast<int64_t>(r) * P + p0 + c] = S[m][n][e];
      }
  if (kLocal && p0 == 0 && cb == 0 && qc == 0) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = (warp * MT + m) * 16 + i * 8 + qr;
        if (r < D) a.part_decay[unit * D + r] = ex2_approx(total[m][i]);
      }
  }
}

// start state of every span from the spans' own contributions: grid (heads, segments, element blocks)
__global__ void gla_span_scan_kernel(const NxGlaArgs a) {
  const int h = blockIdx.x, sg = blockIdx.y;
  const int64_t plane = static_cast<int64_t>(a.dim) * a.vdim;
  const int64_t i = blockIdx.z * static_cast<int64_t>(blockDim.x) + threadIdx.x;
  if (i >= plane) return;
  const int len = a.seg.len[sg], d = static_cast<int>(i / a.vdim);
  float s = a.seg.pos[sg] == 0 ? 0.0f : a.state[(static_cast<int64_t>(a.seg.seq[sg]) * a.heads + h) * plane + i];
  for (int k = 0; k * a.span < len; ++k) {
    const int64_t unit = (static_cast<int64_t>(sg) * a.parts + k) * a.heads + h;
    float* p = a.part_state + unit * plane + i;
    const bool last = (k + 1) * a.span >= len;
    const float own = last ? 0.0f : *p;
    *p = s;
    if (!last) s = a.part_decay[unit * a.dim + d] * s + own;
  }
}

template <int NP>
int launch(const NxGlaArgs* a, cudaStream_t st) {
  constexpr int kBytes = Smem<NP>::kBytes;
  static_assert(kBytes <= 226 * 1024, "shared memory");
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(gla_chunk_kernel<NP, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes) != cudaSuccess ||
        cudaFuncSetAttribute(gla_chunk_kernel<NP, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes) != cudaSuccess)
      return -2;
    once = true;
  }
  const int col_tiles = (a->vdim + kCols - 1) / kCols;
  dim3 grid(a->heads * col_tiles, a->parts, a->seg.count);
  if (a->parts > 1) {
    gla_chunk_kernel<NP, true><<<grid, 256, kBytes, st>>>(*a, col_tiles);
    const int64_t plane = static_cast<int64_t>(a->dim) * a->vdim;
    gla_span_scan_kernel<<<dim3(a->heads, a->seg.count, static_cast<unsigned>((plane + 255) / 256)), 256, 0, st>>>(*a);
  }
  gla_chunk_kernel<NP, false><<<grid, 256, kBytes, st>>>(*a, col_tiles);
  return launch_status();
}

}  // namespace

extern "C" int nx_gla_chunk(const NxGlaArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->dtype != NX_BF16 || a->heads <= 0 || a->dim <= 0 || a->vdim <= 0) return -1;
  if (a->parts < 1 || a->span <= 0 || a->span % kQ) return -1;
  if (a->seg.count <= 0) return 0;
  if (static_cast<int64_t>(a->span) * a->parts < a->seg.max_len || a->seg.count > 65535 || a->parts > 65535) return -1;
  if (a->parts > 1 && (a->part_state == nullptr || a->part_decay == nullptr)) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a->dim <= 64) return launch<64>(a, st);
  if (a->dim <= 128) return launch<128>(a, st);
  if (a->dim <= 256) return launch<256>(a, st);
  return -1;
}
