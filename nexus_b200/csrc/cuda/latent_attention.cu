// Attention over a paged latent cache (see nx_api_mixers.h): all heads share one cache row per token, whose leading columns
// are the values, so a row is read from memory once for every head and for both products.
//
// A block owns 16 MT (token, head) rows of one segment and one span of its keys.  Keys arrive in stages of 32 or 64; the pages of
// a stage come as tiled copies of whole cache rows, split into slabs of 64 columns with the 128-byte swizzle, which the fragment
// loads undo.  The warps split the keys of a stage for the scores and the latent columns for the weighted sum; row maxima and
// probabilities cross warps through shared memory.  Scores and softmax are FP32; only the products take BF16 operands.
#include "flash_common.cuh"
#include "mixer_common.cuh"
#include "nx_api_mixers.h"
#include "paged_common.cuh"
#include "sm100_ptx.cuh"
#include "tensor_map.h"

#include <algorithm>
#include <type_traits>

namespace {
using namespace nx;

constexpr int kKGroups = 4;         // warps along the keys of a stage
constexpr int kBox = 8;             // keys of one copy: what every page size is a multiple of, one row group of the swizzle
constexpr int kSlab = kBox * 128;   // bytes of 64 columns of a box
constexpr int kSmemMax = 226 * 1024;

template <int MT>
struct Shape {
  static constexpr int kRows = 16 * MT;
  static constexpr int kKeys = MT == 2 ? 64 : 32;       // per stage: what shared memory holds twice beside the queries
  static constexpr int kNTiles = kKeys / kKGroups / 8;  // 8-key tiles of a warp
  static constexpr int kLdP = kKeys + 8;
  static constexpr int kMGroups = MT == 1 ? 1 : 2;      // warps along the rows
  static constexpr int kWarps = kKGroups * kMGroups;
  static constexpr int kMTiles = MT / kMGroups;         // 16-row tiles of a warp
  // behind the stages and Q: P, maxima per key group, running maximum, rescale factor, row sums, barriers
  static constexpr int kTail = kRows * kLdP * 2 + kKGroups * kRows * 4 + 3 * kRows * 4 + 128;
};

// CT: 16-column tiles of the latent per warp
template <int MT, int CT>
__global__ void __launch_bounds__(Shape<MT>::kWarps * 32, MT == 1 ? 2 : 1)
latent_attn_kernel(const __grid_constant__ CUtensorMap tm, const NxLatentAttnArgs a, int rt, int tq, int stages) {
  using S = Shape<MT>;
  constexpr int ROWS = S::kRows, WARPS = S::kWarps, THREADS = WARPS * 32, kKeys = S::kKeys, kLdP = S::kLdP, NTILES = S::kNTiles;
  extern __shared__ __align__(1024) uint8_t smem[];
  const int LD = a.row + 8, slabs = a.row / 64, stage_bytes = kKeys * a.row * 2;
  uint8_t* sKV = smem;                                                // [stages][boxes][slabs][kBox][128 B]
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem + stages * stage_bytes);   // [ROWS][LD]
  __nv_bfloat16* sP = sQ + ROWS * LD;                                 // [ROWS][kLdP]
  float* s_part = reinterpret_cast<float*>(sP + ROWS * kLdP);         // [key groups][ROWS] stage maxima, then row sums
  float* s_max = s_part + kKGroups * ROWS;                            // running maximum of a row (log2 units)
  float* s_alpha = s_max + ROWS;
  float* s_sum = s_alpha + ROWS;
  uint64_t* full = reinterpret_cast<uint64_t*>(s_sum + ROWS);         // [stages]
  uint64_t* empty = full + stages;                                    // [stages], one arrival per warp
  __shared__ int s_tile[3];
  __shared__ volatile int s_abort;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  if (smem_u32(smem) & 1023u) {   // the swizzle needs a 1 KiB aligned base; uniform early exit
    if (threadIdx.x == 0) atomicCAS(a.status, 0, kStatusBadArgument);
    return;
  }
  if (warp == 0) {
    int seg = 0, off = 0;
    const bool ok = find_tile(a.seg, tq, blockIdx.x, seg, off);
    if (lane == 0) {
      s_tile[0] = ok;
      s_tile[1] = seg;
      s_tile[2] = off;
      s_abort = 0;
      for (int i = 0; i < stages; ++i) {
        mbar_init(&full[i], 1);
        mbar_init(&empty[i], WARPS);
      }
      fence_mbar_init();
    }
  }
  __syncthreads();
  if (!s_tile[0]) return;
  const int sg = s_tile[1], t0 = s_tile[2] * tq, h0 = blockIdx.y * rt;
  const int nh = min(rt, a.heads - h0), nt = min(tq, a.seg.len[sg] - t0), pos0 = a.seg.pos[sg] + t0;
  const int64_t row0 = static_cast<int64_t>(a.seg.row0[sg]) + t0;
  const int hi = pos0 + nt - 1, lo = (a.window > 0 ? max(0, pos0 - a.window + 1) : 0) & ~(kBox - 1);
  const int per = ((hi - lo + kKeys) / kKeys + a.splits - 1) / a.splits * kKeys;
  const int first = lo + static_cast<int>(blockIdx.z) * per, last = min(hi, first + per - 1);
  const int n_stages = last >= first ? (last - first) / kKeys + 1 : 0;
  const int32_t* bt = a.block_table + static_cast<int64_t>(a.seg.seq[sg]) * a.max_blocks;
  const int shift = log2_of(a.block_size);
  // boxes past the last key repeat the last one (masked below), so that every row of a stage holds finite values
  auto load = [&](int it) {
    if (threadIdx.x != 0) return;
    const int s = it % stages;
    mbar_arrive_expect_tx(&full[s], static_cast<uint32_t>(stage_bytes));
    int slot[kKeys / kBox];
#pragma unroll
    for (int b = 0; b < kKeys / kBox; ++b)
      slot[b] = static_cast<int>(page_slot(bt, a.block_size, shift, min(first + it * kKeys + b * kBox, hi & ~(kBox - 1))));
#pragma unroll
    for (int b = 0; b < kKeys / kBox; ++b)
      tma_load_3d(sKV + s * stage_bytes + b * slabs * kSlab, &tm, &full[s], 0, slot[b], 0);
  };
  for (int it = 0; it < min(stages, n_stages); ++it) load(it);
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q);
    const int ch = a.row / 8;
    for (int m = warp; m < ROWS; m += WARPS) {
      const int tok = m / rt, hh = m % rt;
      const bool in = tok < nt && hh < nh;
      const uint4* src = reinterpret_cast<const uint4*>(q + (row0 + tok) * a.ldq + static_cast<int64_t>(h0 + hh) * a.row);
      for (int c = lane; c < ch; c += 32)
        *reinterpret_cast<uint4*>(sQ + m * LD + c * 8) = in ? src[c] : make_uint4(0u, 0u, 0u, 0u);
    }
  }
  for (int m = threadIdx.x; m < ROWS; m += THREADS) s_max[m] = -INFINITY;
  const int mg = warp % S::kMGroups, kg = warp / S::kMGroups;
  const float mul = a.scale * kLog2e;
  int vis[S::kMTiles][2];                           // position of this thread's score rows, -1: padding row
  float sum[S::kMTiles][2], ref[S::kMTiles][2];     // ref: what the row's scores are measured against (log2 units)
  const bool full_tile = nt * rt == ROWS && nh == rt;
#pragma unroll
  for (int i = 0; i < S::kMTiles; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int m = (mg * S::kMTiles + i) * 16 + e * 8 + g;
      vis[i][e] = m / rt < nt && m % rt < nh ? pos0 + m / rt : -1;
      sum[i][e] = 0.0f;
      ref[i][e] = -INFINITY;
    }
  float o[MT][CT][2][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int c = 0; c < CT; ++c)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[i][c][0][e] = o[i][c][1][e] = 0.0f;
  // byte offset of a key row inside a stage (slab 0); its 16-byte chunks are swizzled by the key
  auto key_offset = [&](int key) -> uint32_t { return (key / kBox) * slabs * kSlab + (key % kBox) * 128; };
  uint32_t k_off[NTILES];
#pragma unroll
  for (int n = 0; n < NTILES; ++n) k_off[n] = key_offset((kg * NTILES + n) * 8 + (lane & 7)) + (((lane >> 3) ^ (lane & 7)) << 4);
  // value fragments: this warp's first 16 columns; a round of the warps is WARPS / 4 slabs
  const uint32_t v_col = (warp >> 2) * kSlab + ((((warp & 3) * 2 + (lane >> 4)) ^ (lane & 7)) << 4);
  uint32_t v_off[kKeys / 16];
#pragma unroll
  for (int kk = 0; kk < kKeys / 16; ++kk) v_off[kk] = key_offset(kk * 16 + (lane & 15)) + v_col;
  const int rounds = (a.rank + WARPS * 16 - 1) / (WARPS * 16);
  const uint32_t q_addr = smem_addr(sQ + (mg * S::kMTiles * 16 + (lane & 15)) * LD + (lane >> 4) * 8);
  __syncthreads();
  bool ok = true;
  for (int it = 0; it < n_stages; ++it) {
    const int s = it % stages, k0 = first + it * kKeys;
    if (threadIdx.x == 0 && it > 0 && it - 1 + stages < n_stages) {     // the stage of the previous round, once all have used it
      ok = ok && mbar_wait_bounded(&empty[(it - 1) % stages], ((it - 1) / stages) & 1, &s_abort);
      if (ok) load(it - 1 + stages);
    }
    ok = ok && mbar_wait_bounded(&full[s], (it / stages) & 1, &s_abort);
    const uint32_t base = smem_u32(sKV) + s * stage_bytes;
    // partial sums over the columns, so that few products wait for one another
    constexpr int CHAINS = S::kMTiles * NTILES == 1 ? 4 : 2;
    float part[CHAINS][S::kMTiles][NTILES][4];
#pragma unroll
    for (int c = 0; c < CHAINS; ++c)
#pragma unroll
      for (int i = 0; i < S::kMTiles; ++i)
#pragma unroll
        for (int n = 0; n < NTILES; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) part[c][i][n][e] = 0.0f;
    // the fragments of the next slab are on their way while this one's products run
    uint32_t kf[2][NTILES][2][4], qf[2][S::kMTiles][4][4];
    auto fetch = [&](uint32_t slab, uint32_t q, int u) {
#pragma unroll
      for (int n = 0; n < NTILES; ++n) {
        ldmatrix_x4(kf[u][n][0], slab + k_off[n]);
        ldmatrix_x4(kf[u][n][1], (slab + k_off[n]) ^ 64);          // columns 32..63: the other half of the 128 bytes
      }
#pragma unroll
      for (int i = 0; i < S::kMTiles; ++i)
#pragma unroll
        for (int c = 0; c < 4; ++c) ldmatrix_x4(qf[u][i][c], q + i * 32 * LD + c * 32);
    };
    auto multiply = [&](int u) {
#pragma unroll
      for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int i = 0; i < S::kMTiles; ++i)
#pragma unroll
          for (int n = 0; n < NTILES; ++n)
            mma_bf16(part[c % CHAINS][i][n], qf[u][i][c], kf[u][n][c >> 1][(c & 1) * 2], kf[u][n][c >> 1][(c & 1) * 2 + 1]);
    };
    uint32_t slab = base, qs = q_addr;
    fetch(slab, qs, 0);
    int b = 0;
    for (; b + 2 < slabs; b += 2, slab += 2 * kSlab, qs += 256) {
      fetch(slab + kSlab, qs + 128, 1);
      multiply(0);
      fetch(slab + 2 * kSlab, qs + 256, 0);
      multiply(1);
    }
    if (b + 1 < slabs) fetch(slab + kSlab, qs + 128, 1);
    multiply(0);
    if (b + 1 < slabs) multiply(1);
    float sc[S::kMTiles][NTILES][4];
#pragma unroll
    for (int i = 0; i < S::kMTiles; ++i)
#pragma unroll
      for (int n = 0; n < NTILES; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          sc[i][n][e] = part[0][i][n][e] + part[1][i][n][e];
          if constexpr (CHAINS == 4) sc[i][n][e] += part[2][i][n][e] + part[3][i][n][e];
          sc[i][n][e] *= mul;
        }
    const int kbase = k0 + kg * NTILES * 8 + t * 2;
    const bool inside = k0 + kKeys - 1 <= min(pos0, last) && (a.window <= 0 || k0 > hi - a.window) && full_tile;
    float top[S::kMTiles][2];
    bool grow = false;
#pragma unroll
    for (int i = 0; i < S::kMTiles; ++i) {
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int n = 0; n < NTILES; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (!inside) {                              // some row of the block does not see the whole stage
            const int j = kbase + n * 8 + (e & 1), p = vis[i][e >> 1];
            if (!(j <= min(p, last) && (a.window <= 0 || j > p - a.window))) sc[i][n][e] = -INFINITY;
          }
          mx[e >> 1] = fmaxf(mx[e >> 1], sc[i][n][e]);
        }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        top[i][e] = mx[e];
        grow = grow || mx[e] > ref[i][e] + kRescaleStep;
      }
    }
    // every warp weighs with one reference per row; it moves only when a row's maximum has grown by 2^8.  Past this barrier
    // every warp is done with the previous P, too.
    const bool move = __syncthreads_or(grow) != 0;
    if (move) {
#pragma unroll
      for (int i = 0; i < S::kMTiles; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float mx = fmaxf(top[i][e], __shfl_xor_sync(0xffffffffu, top[i][e], 1));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
          if (t == 0) s_part[kg * ROWS + (mg * S::kMTiles + i) * 16 + e * 8 + g] = mx;
        }
      __syncthreads();
      if (threadIdx.x < ROWS) {
        const int m = threadIdx.x;
        const float old = s_max[m];
        float nm = old;
#pragma unroll
        for (int w = 0; w < kKGroups; ++w) nm = fmaxf(nm, s_part[w * ROWS + m]);
        const bool up = nm > old + kRescaleStep;
        s_alpha[m] = up ? ex2_approx(old - nm) : 1.0f;
        if (up) s_max[m] = nm;
      }
      __syncthreads();
#pragma unroll
      for (int i = 0; i < S::kMTiles; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int m = (mg * S::kMTiles + i) * 16 + e * 8 + g;
          ref[i][e] = s_max[m];
          sum[i][e] *= s_alpha[m];
        }
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const float f0 = s_alpha[i * 16 + g], f1 = s_alpha[i * 16 + 8 + g];
#pragma unroll
        for (int c = 0; c < CT; ++c)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            o[i][c][n][0] *= f0;
            o[i][c][n][1] *= f0;
            o[i][c][n][2] *= f1;
            o[i][c][n][3] *= f1;
          }
      }
    }
#pragma unroll
    for (int i = 0; i < S::kMTiles; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int m = (mg * S::kMTiles + i) * 16 + e * 8 + g;
        const float base_m = ref[i][e] == -INFINITY ? 0.0f : ref[i][e];
#pragma unroll
        for (int n = 0; n < NTILES; ++n) {
          const float p0 = ex2_approx(sc[i][n][2 * e] - base_m), p1 = ex2_approx(sc[i][n][2 * e + 1] - base_m);   // -inf: 0
          sum[i][e] += p0 + p1;
          *reinterpret_cast<uint32_t*>(sP + m * kLdP + (kg * NTILES + n) * 8 + t * 2) = bf16_pair(p0, p1);
        }
      }
    __syncthreads();
    // columns past the latent (a last, partial round of tiles) are multiplied but not stored
    auto weigh = [&](auto tiles, int n) {
      constexpr int N = decltype(tiles)::value;
#pragma unroll
      for (int kk = 0; kk < kKeys / 16; ++kk) {
        uint32_t pa[MT][4], vb[N][4];
#pragma unroll
        for (int i = 0; i < MT; ++i)
          ldmatrix_x4(pa[i], smem_addr(sP + (i * 16 + (lane & 15)) * kLdP + kk * 16 + (lane >> 4) * 8));
#pragma unroll
        for (int c = 0; c < N; ++c)
          if (N == CT || c < n) ldmatrix_x4_trans(vb[c], base + v_off[kk] + c * (WARPS / 4) * kSlab);
#pragma unroll
        for (int c = 0; c < N; ++c)
          if (N == CT || c < n) {
#pragma unroll
            for (int i = 0; i < MT; ++i) {
              mma_bf16(o[i][c][0], pa[i], vb[c][0], vb[c][1]);
              mma_bf16(o[i][c][1], pa[i], vb[c][2], vb[c][3]);
            }
          }
      }
    };
    if (rounds == CT) weigh(std::integral_constant<int, CT>{}, CT);
    else if constexpr (CT > 1) weigh(std::integral_constant<int, CT - 1>{}, rounds);
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[s]);
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < S::kMTiles; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      sum[i][e] += __shfl_xor_sync(0xffffffffu, sum[i][e], 1);
      sum[i][e] += __shfl_xor_sync(0xffffffffu, sum[i][e], 2);
      if (t == 0) s_part[kg * ROWS + (mg * S::kMTiles + i) * 16 + e * 8 + g] = sum[i][e];
    }
  __syncthreads();
  if (threadIdx.x < ROWS) {
    float l = 0.0f;
#pragma unroll
    for (int w = 0; w < kKGroups; ++w) l += s_part[w * ROWS + threadIdx.x];
    s_sum[threadIdx.x] = l;
  }
  __syncthreads();
  if (!ok) {
    // a wait ran out: time for copies still in flight to land before the shared memory goes away
    atomicCAS(a.status, 0, kStatusTimeoutProducer);
    const uint64_t begin = globaltimer_ns();
    while (globaltimer_ns() - begin < 2000000ull) __nanosleep(2000);
  }
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int m = i * 16 + e * 8 + g, tok = m / rt, h = h0 + m % rt;
      if (tok >= nt || m % rt >= nh) continue;
      const int64_t r = row0 + tok;
      if (a.splits == 1) {
        const float f = (a.gate != nullptr ? a.gate[r * a.heads + h] : 1.0f) / s_sum[m];
        __nv_bfloat16* op = static_cast<__nv_bfloat16*>(a.out) + r * a.ldo + static_cast<int64_t>(h) * a.rank;
#pragma unroll
        for (int c = 0; c < CT; ++c)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const int col = (c * WARPS + warp) * 16 + n * 8 + t * 2;
            if (col < a.rank) *reinterpret_cast<uint32_t*>(op + col) = bf16_pair(o[i][c][n][2 * e] * f, o[i][c][n][2 * e + 1] * f);
          }
      } else {
        const int64_t pi = (r * a.heads + h) * a.splits + blockIdx.z;
#pragma unroll
        for (int c = 0; c < CT; ++c)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const int col = (c * WARPS + warp) * 16 + n * 8 + t * 2;
            if (col < a.rank)
              *reinterpret_cast<float2*>(a.part_o + pi * a.rank + col) = make_float2(o[i][c][n][2 * e], o[i][c][n][2 * e + 1]);
          }
        if (warp == 0 && t == 0) {
          a.part_ml[pi * 2] = s_max[m];
          a.part_ml[pi * 2 + 1] = s_sum[m];
        }
      }
    }
}

// one block per (segment row, head): the spans of its keys
__global__ void latent_merge_kernel(const NxLatentAttnArgs a) {
  const int sg = blockIdx.z, t = blockIdx.x, h = blockIdx.y;
  if (t >= a.seg.len[sg]) return;
  const int64_t r = static_cast<int64_t>(a.seg.row0[sg]) + t, base = (r * a.heads + h) * a.splits;
  float gm = -INFINITY, gl = 0.0f;
  for (int s = 0; s < a.splits; ++s) gm = fmaxf(gm, a.part_ml[(base + s) * 2]);
  for (int s = 0; s < a.splits; ++s) {
    const float m = a.part_ml[(base + s) * 2];
    gl += m == -INFINITY ? 0.0f : a.part_ml[(base + s) * 2 + 1] * exp2f(m - gm);
  }
  const float f = (a.gate != nullptr ? a.gate[r * a.heads + h] : 1.0f) / gl;
  for (int d = threadIdx.x * 4; d < a.rank; d += blockDim.x * 4) {
    float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    for (int s = 0; s < a.splits; ++s) {
      const float m = a.part_ml[(base + s) * 2], w = m == -INFINITY ? 0.0f : exp2f(m - gm) * f;
      const float4 p = *reinterpret_cast<const float4*>(a.part_o + (base + s) * a.rank + d);
      v.x += p.x * w;
      v.y += p.y * w;
      v.z += p.z * w;
      v.w += p.w * w;
    }
    *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(a.out) + r * a.ldo + static_cast<int64_t>(h) * a.rank + d) =
        make_uint2(bf16_pair(v.x, v.y), bf16_pair(v.z, v.w));
  }
}

template <int MT, int CT>
int launch(const CUtensorMap& tm, const NxLatentAttnArgs* a, cudaStream_t st) {
  using S = Shape<MT>;
  const int stage = S::kKeys * a->row * 2, fixed = S::kRows * (a->row + 8) * 2 + S::kTail;
  // two blocks per SM where two stages fit twice, else one block with a deeper ring
  const int half = (kSmemMax / 2 - 1024 - fixed) / stage;
  const int stages = std::min(4, half >= 2 ? half : (kSmemMax - 1024 - fixed) / stage);
  if (stages < 2) return -1;
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(latent_attn_kernel<MT, CT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemMax - 1024) != cudaSuccess)
      return -2;
    once = true;
  }
  const int rt = std::min(a->heads, S::kRows), tq = std::max(1, S::kRows / rt);
  const dim3 grid(a->seg.total_len / tq + a->seg.count, (a->heads + rt - 1) / rt, a->splits);
  latent_attn_kernel<MT, CT><<<grid, S::kWarps * 32, fixed + stages * stage, st>>>(tm, *a, rt, tq, stages);
  return launch_status();
}

template <int MT>
int launch_rank(const CUtensorMap& tm, const NxLatentAttnArgs* a, cudaStream_t st) {
  constexpr int kW = Shape<MT>::kWarps;
  if (a->rank <= 128) return launch<MT, 8 / kW>(tm, a, st);
  if (a->rank <= 256) return launch<MT, 16 / kW>(tm, a, st);
  return launch<MT, 32 / kW>(tm, a, st);
}

}  // namespace

extern "C" int nx_latent_attention(const NxLatentAttnArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->status == nullptr || a->heads <= 0 || a->rank <= 0 || a->rank > 512 || (a->rank & 15)) return -1;
  if (a->row < a->rank || (a->row & 63) || a->row > 768 || a->block_size < 8 || (a->block_size & 7)) return -1;
  if (a->max_blocks <= 0 || a->splits < 1 || a->n_slots <= 0) return -1;
  if (a->splits > 1 && (a->part_o == nullptr || a->part_ml == nullptr)) return -1;
  if ((a->ldq & 7) || (a->ldo & 7) || a->seg.count > 65535 || a->splits > 65535) return -1;
  if ((reinterpret_cast<uintptr_t>(a->q) & 15) || (reinterpret_cast<uintptr_t>(a->cache) & 15)) return -1;
  if (a->seg.count <= 0 || a->seg.max_len <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  CUtensorMap tm;
  {
    // {64 columns, cache slots, slabs}: one copy brings whole rows, slab by slab
    nx::EncodeTiledFn fn = nx::encode_tiled_fn();
    if (fn == nullptr) return -3;
    const cuuint32_t slabs = static_cast<cuuint32_t>(a->row / 64);
    cuuint64_t dims[3] = {64, static_cast<cuuint64_t>(a->n_slots), slabs}, strides[2] = {static_cast<cuuint64_t>(a->row) * 2, 128};
    cuuint32_t box[3] = {64, kBox, slabs}, one[3] = {1, 1, 1};
    if (fn(&tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(a->cache), dims, strides, box, one,
           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
      return -4;
  }
  const int rows = a->seg.max_len > 1 ? 64 : a->heads;      // (token, head) pairs of a block
  const int rc = rows <= 16 ? launch_rank<1>(tm, a, st)
                 : rows <= 32 && a->row <= 640 ? launch_rank<2>(tm, a, st) : launch_rank<4>(tm, a, st);
  if (rc == 0 && a->splits > 1) {
    latent_merge_kernel<<<dim3(a->seg.max_len, a->heads, a->seg.count), std::min(128, (a->rank / 4 + 31) / 32 * 32), 0, st>>>(*a);
    return launch_status();
  }
  return rc;
}
