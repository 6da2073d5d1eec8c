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
// The ten 16 x 16 blocks of the inner sums are shared out among the warps and pass through shared memory.  Only F_ii grows with the
// decay.  Where a sub-block decays by more than 2^60 its own products are formed pair by pair from the exponents' differences
// instead, so any decay is exact.
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
constexpr int kBlocks = 10;            // (sub-block, earlier or same sub-block): block i (i + 1) / 2 + j

template <int NP>
struct Smem {
  static constexpr int LN = NP + 8, LP = kCols + 8;
  static constexpr int kQh = 0, kQl = kQh + kQ * LN, kKh = kQl + kQ * LN, kKl = kKh + kQ * LN, kV = kKl + kQ * LN,
                       kSh = kV + kQ * LP, kSl = kSh + NP * LP, kEnd = kSl + NP * LP;
  // the blocks of token products lie over q, whose last use is before theirs, where the rest leaves no room
  static constexpr bool kOverQ = kEnd * 2 + 8 * NP * 4 + kBlocks * 1024 > 226 * 1024;
  static constexpr int kBytes = kEnd * 2 + 8 * NP * 4 + (kOverQ ? 0 : kBlocks * 1024);
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

// G = (q of sub-block i, times `f` per channel where `scaled`) k^T of sub-block j, pairs of BF16
template <int NP, typename Factor>
__device__ __forceinline__ void block_product(float (&g)[2][4], const __nv_bfloat16* sQh, const __nv_bfloat16* sQl,
                                              const __nv_bfloat16* sKh, const __nv_bfloat16* sKl, int i, int j, bool scaled, Factor factor) {
  constexpr int LN = Smem<NP>::LN;
#pragma unroll
  for (int kk = 0; kk < NP / 16; ++kk) {
    uint32_t qh[4], ql[4], bh[4], bl[4];
    ldmatrix_x4(qh, addr_a<LN>(sQh, i * kSub, kk * 16));
    ldmatrix_x4(ql, addr_a<LN>(sQl, i * kSub, kk * 16));
    ldmatrix_x4(bh, addr_b<LN>(sKh, j * kSub, kk * 16));
    ldmatrix_x4(bl, addr_b<LN>(sKl, j * kSub, kk * 16));
    if (scaled) {
      float f[4];
      factor(kk, f);
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
  float* sD = reinterpret_cast<float*>(sm + L::kEnd);    // [4][NP]: 2^R of every sub-block
  float* sI = sD + 4 * NP;                               // [4][NP]: 2^-R
  uint4* sG = L::kOverQ ? reinterpret_cast<uint4*>(sQh) : reinterpret_cast<uint4*>(sI + 4 * NP);   // [kBlocks][hi, lo][lane]
  __shared__ int s_far[2][4];                            // sub-blocks whose decay is not inverted, by chunk parity
  const int h = blockIdx.x / col_tiles, p0 = (blockIdx.x % col_tiles) * kCols, part = blockIdx.y, sg = blockIdx.z;
  const int len = a.seg.len[sg], t_begin = part * a.span, t_end = min(len, t_begin + a.span);
  if (t_begin >= len || (kLocal && t_end == len)) return;   // the last span's contribution is never needed
  const int D = a.dim, P = a.vdim, cols = min(kCols, P - p0);
  const int wid = threadIdx.x >> 5, warp = wid & 3, cb = (wid >> 2) * 32, lane = threadIdx.x & 31, qr = lane >> 2, qc = (lane & 3) * 2;
  const int64_t row0 = a.seg.row0[sg];
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + row0 * a.ld + static_cast<int64_t>(h) * D;
  const __nv_bfloat16* k = static_cast<const __nv_bfloat16*>(a.k) + row0 * a.ld + static_cast<int64_t>(h) * D;
  const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(a.v) + row0 * a.ld + static_cast<int64_t>(h) * P + p0;
  const float* dec = a.decay + row0 * a.ld_decay + static_cast<int64_t>(h) * D;
  const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec_d = (a.ld & 7) == 0 && (D & 7) == 0 && al(a.q) && al(a.k), vec_p = (a.ld & 7) == 0 && (P & 7) == 0 && al(a.v);
  const bool vec_a = (a.ld_decay & 1) == 0 && (D & 1) == 0 && al(a.decay);
  const int64_t plane = static_cast<int64_t>(D) * P;
  float* pool = a.state + (static_cast<int64_t>(a.seg.seq[sg]) * a.heads + h) * plane;
  const int64_t unit = (static_cast<int64_t>(sg) * a.parts + part) * a.heads + h;
  float* part_state = a.parts > 1 ? a.part_state + unit * plane : nullptr;
  float S[MT][4][4], total[MT][2];                       // total: decay of the span
  {
    const float* src = kLocal ? nullptr : a.parts > 1 ? part_state : (a.seg.pos[sg] == 0 ? nullptr : pool);
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      total[m][0] = total[m][1] = 1.0f;
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
  // Log2 decays of the chunk to convert next.  A warp takes one sub-block and 16 pairs of channels; lanes 16-31 hold the
  // sub-block's last eight tokens.
  const int half = lane >> 4;
  float raw[ITEMS][8][2];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int item = wid + i * 8, d = (item % (NP / 32)) * 32 + (lane & 15) * 2, t = t0 + item / (NP / 32) * kSub + half * 8;
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const float* p = dec + static_cast<int64_t>(t + u) * a.ld_decay + d;
        float2 x = make_float2(0.0f, 0.0f);
        if (t + u < t_end) {
          if (vec_a) {
            if (d < D) x = *reinterpret_cast<const float2*>(p);
          } else {
            if (d < D) x.x = p[0];
            if (d + 1 < D) x.y = p[1];
          }
        }
        raw[i][u][0] = x.x;
        raw[i][u][1] = x.y;
      }
    }
  };
  auto scale_store = [&](__nv_bfloat16* hi, __nv_bfloat16* lo, int o, float f0, float f1) {
    const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(hi + o);
    uint32_t xh, xl;
    bf16_split(__low2float(x) * f0, __high2float(x) * f1, xh, xl);
    *reinterpret_cast<uint32_t*>(hi + o) = xh;
    *reinterpret_cast<uint32_t*>(lo + o) = xl;
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
      const int item = wid + i * 8, d = (item % (NP / 32)) * 32 + (lane & 15) * 2, j = item / (NP / 32);
      float before[2], end[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
#pragma unroll
        for (int u = 1; u < 8; ++u) raw[i][u][e] += raw[i][u - 1][e];
        const float other = __shfl_xor_sync(0xffffffffu, raw[i][7][e], 16);
        before[e] = half ? other : 0.0f;
        end[e] = raw[i][7][e] + other;
      }
      if (half == 0) {
        *reinterpret_cast<float2*>(sD + j * NP + d) = make_float2(ex2_approx(end[0]), ex2_approx(end[1]));
        *reinterpret_cast<float2*>(sI + j * NP + d) = make_float2(ex2_approx(-end[0]), ex2_approx(-end[1]));
        if (fminf(end[0], end[1]) < kSafe) s_far[par][j] = 1;
      }
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        // the halves of a warp are four rows apart in the walk, which keeps their banks apart
        const float c0 = (half ? raw[i][u ^ 4][0] : raw[i][u][0]) + before[0], c1 = (half ? raw[i][u ^ 4][1] : raw[i][u][1]) + before[1];
        const int o = (j * kSub + half * 8 + (half ? u ^ 4 : u)) * LN + d;
        if (!kLocal) scale_store(sQh, sQl, o, a.q_scale * ex2_approx(c0), a.q_scale * ex2_approx(c1));
        scale_store(sKh, sKl, o, ex2_approx(end[0] - c0), ex2_approx(end[1] - c1));
      }
    }
    if (more) fetch(t0 + kQ);
    __syncthreads();
    if (threadIdx.x < 4) s_far[par ^ 1][threadIdx.x] = 0;
    if (!kLocal) {
      // the lane's four channels of the product of the decays of sub-blocks j0 .. j1 - 1
      auto decays = [&](int kk, int j0, int j1, float (&f)[4]) {
        f[0] = f[1] = f[2] = f[3] = 1.0f;
        for (int j = j0; j < j1; ++j) {
          const float2 x = *reinterpret_cast<const float2*>(sD + j * NP + kk * 16 + qc);
          const float2 y = *reinterpret_cast<const float2*>(sD + j * NP + kk * 16 + 8 + qc);
          f[0] *= x.x;
          f[1] *= x.y;
          f[2] *= y.x;
          f[3] *= y.y;
        }
      };
      auto inner = [&](int i, int j, float (&g)[2][4]) {
        zero(g);
        if (j < i) {
          block_product<NP>(g, sQh, sQl, sKh, sKl, i, j, j + 1 < i, [&](int kk, float (&f)[4]) { decays(kk, j + 1, i, f); });
          return;
        }
        if (s_far[par][i]) {
          // the decay between two tokens directly: lane t < 16 holds token t of the sub-block
          const int t = t0 + i * kSub + (lane & 15);
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
          block_product<NP>(g, sQh, sQl, sKh, sKl, i, i, true, [&](int kk, float (&f)[4]) {
            const float2 x = *reinterpret_cast<const float2*>(sI + i * NP + kk * 16 + qc);
            const float2 y = *reinterpret_cast<const float2*>(sI + i * NP + kk * 16 + 8 + qc);
            f[0] = x.x;
            f[1] = x.y;
            f[2] = y.x;
            f[3] = y.y;
          });
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (n * 8 + qc + (e & 1) > (e >> 1) * 8 + qr) g[n][e] = 0.0f;
      };
      auto put = [&](int i, int j, const float (&g)[2][4]) {
        uint4 hi, lo;
        bf16_split(g[0][0], g[0][1], hi.x, lo.x);
        bf16_split(g[0][2], g[0][3], hi.y, lo.y);
        bf16_split(g[1][0], g[1][1], hi.z, lo.z);
        bf16_split(g[1][2], g[1][3], hi.w, lo.w);
        uint4* dst = sG + (i * (i + 1) / 2 + j) * 64 + lane;
        dst[0] = hi;
        dst[32] = lo;
      };
      // Ten blocks on eight warps: the three next to the diagonal need no factors, so two warps take two blocks.
      //   warp   0      1      2             3      4      5             6      7
      //   block  (3,0)  (3,1)  (3,2), (0,0)  (3,3)  (2,0)  (2,1), (1,0)  (2,2)  (1,1)
      const int bi = wid < 4 ? 3 : wid < 7 ? 2 : 1, bj = wid < 4 ? wid : wid < 7 ? wid - 4 : 1;
      float g0[2][4], g1[2][4];
      inner(bi, bj, g0);
      if (wid == 2) inner(0, 0, g1);
      if (wid == 5) inner(1, 0, g1);
      float y[4][4];
      zero(y);
#pragma unroll
      for (int kk = 0; kk < NP / 16; ++kk) {             // q S
        uint32_t qh[4], ql[4];
        ldmatrix_x4(qh, addr_a<LN>(sQh, warp * kSub, kk * 16));
        ldmatrix_x4(ql, addr_a<LN>(sQl, warp * kSub, kk * 16));
        if (warp > 0) {
          float f[4];
          decays(kk, 0, warp, f);
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
      if constexpr (L::kOverQ) __syncthreads();          // q has been read
      put(bi, bj, g0);
      if (wid == 2) put(0, 0, g1);
      if (wid == 5) put(1, 0, g1);
      __syncthreads();                                   // the blocks are complete; q is free
      if (!L::kOverQ && more) load_q(t0 + kQ);
      for (int j = 0; j <= warp; ++j) {
        const uint4* src = sG + (warp * (warp + 1) / 2 + j) * 64 + lane;
        const uint4 hi = src[0], lo = src[32];
        const uint32_t mh[4] = {hi.x, hi.y, hi.z, hi.w}, ml[4] = {lo.x, lo.y, lo.z, lo.w};
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, addr_b_t<LP>(sV, j * kSub, cb + n * 16));
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
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      uint32_t kh[MT][4], kl[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const int r = (warp * MT + m) * 16;
        ldmatrix_x4_trans(kh[m], addr_a_t<LN>(sKh, j * kSub, r));
        ldmatrix_x4_trans(kl[m], addr_a_t<LN>(sKl, j * kSub, r));
        const float d0 = sD[j * NP + r + qr], d1 = sD[j * NP + r + 8 + qr];
        total[m][0] *= d0;
        total[m][1] *= d1;
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
        ldmatrix_x4_trans(b, addr_b_t<LP>(sV, j * kSub, cb + n * 16));
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
      if (L::kOverQ && !kLocal) load_q(t0 + kQ);
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
        if (r < D) a.part_decay[unit * D + r] = total[m][i];
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
  static_assert(kBytes <= 227 * 1024 - 64, "shared memory");
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
