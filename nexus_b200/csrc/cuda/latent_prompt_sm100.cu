// Attention of prompt segments on tcgen05 (see nx_api_mixers.h).  A key is a part of its own KV head, optionally beside a part
// that all heads share; a row sees a window of keys and optionally the first keys of its sequence; a sink may count in the
// denominator.  Queries, keys and values of all segments lie packed in row buffers; a work item is a block of up to 256 query
// rows of one segment and one head.  Without a shared key part a row may also see only the keys of its own chunk of positions, scores
// may have a bias by distance.
//
// The pipeline is that of the two-tile flash kernel: one persistent CTA per SM, softmax group A (warps 0-3) on query rows
// 0-127 of the block, group B (warps 4-7) on rows 128-255, both against the same key tiles; the MMA warp interleaves
//   PV_A(j-1), QK_A(j), PV_B(j-1), QK_B(j).
// S and O live in TMEM (S_A 0-127, S_B 128-255, O_A 256.., O_B 384..); the probabilities go back as BF16 into the columns of
// their score tile and are the A operand of P V from there.  O is rescaled only when a row's maximum has grown by 2^8.
// Key tiles start at the first key the block can see: with a window no tile is wasted on keys before it.  Kept first keys that
// lie before the window come first, in tiles of their own.  Keys and values have rings of their own, since a key part of 192
// columns leaves room for one stage of values.
#include "flash_common.cuh"
#include "nx_api_mixers.h"
#include "sm100_ptx.cuh"
#include "tensor_map.h"

#include <algorithm>

namespace {
using namespace nx;

constexpr int kThreads = 320;   // warps 0-3: softmax A, 4-7: softmax B, 8: TMA, 9: MMA
constexpr int kSlab = 128 * 128;  // bytes of [128 rows][64 columns]

// distances of a bias table in shared memory, and how far it goes on to the masked ones (a row and a key of one tile pair are up to 254
// apart in the wrong direction) and beyond the last one
constexpr int kBiasMax = 3072, kBiasNear = 256, kBiasFar = 256, kBiasTable = kBiasNear + kBiasMax + kBiasFar;

// ND / NV: 64-column slabs of a head's own key part and of its values; NR: of the shared part (0 or 1)
// kBias: a table of biases per softmax group behind the barriers
template <int ND, int NR, int NV, bool kBias>
struct Cfg {
  static constexpr int kQBytes = (ND + NR) * kSlab;
  static constexpr int kKBytes = (ND + NR) * kSlab;
  static constexpr int kVBytes = NV * kSlab;
  static constexpr int kKStages = 2;
  static constexpr int kVStages = 2 * kQBytes + 2 * kKBytes + 2 * kVBytes <= 224 * 1024 ? 2 : 1;
  static constexpr int kSmem = 2 * kQBytes + kKStages * kKBytes + kVStages * kVBytes + 256 + (kBias ? 2 * kBiasTable * 4 : 0);
  static_assert(kSmem <= 227 * 1024, "shared memory");
};

struct Dev {
  const int32_t* blocks;     // [n_blocks][4]: first row, rows, position of the first row, buffer row of position 0
  const int32_t* kept;       // [n_blocks]: buffer row that position 0 has among the kept keys; null: as for the others
  __nv_bfloat16* out;
  const float* gate;
  const float* sink;
  int* status;
  int64_t ldo;
  const float* bias;         // [heads][bias_len]
  int items, heads, rep, vdim, window, keep_first, ksteps, rsteps;   // rep: query heads per KV head; 16-column steps of the own
  int chunk, bias_len;                                               // and the shared key part
  float scale;
  __device__ __forceinline__ int first_key(int pos) const {          // apart from the kept ones
    const int lo = window > 0 ? max(0, pos - window + 1) : 0;
    return chunk > 0 ? max(lo, pos / chunk * chunk) : lo;
  }
};

struct Work {
  int h, row0, rows, pos0, kv0, k_lo;
  int kept0, n_kept;               // buffer row of kept key 0; kept keys before k_lo
  int shift;                       // key tile j < shift holds kept keys 128 j .., tile j >= shift keys k_lo + 128 (j - shift) ..
  int jbA, jeA, jbB, jeB, je;      // key tiles of either query tile
  __device__ __forceinline__ int first_key(int j) const { return j < shift ? j * 128 : k_lo + (j - shift) * 128; }
};
// kKeep: rows may keep first keys (the forms without a shared key part).  CTA c takes items round * grid + c in even rounds and from the other end in odd ones; blocks are sorted by cost
template <bool kKeep>
__device__ __forceinline__ bool next_work(const Dev& p, int round, Work& w) {
  const int G = static_cast<int>(gridDim.x), c = static_cast<int>(blockIdx.x);
  const int item = round * G + ((round & 1) ? (G - 1 - c) : c);
  if (item >= p.items) return false;
  const int4 b = __ldg(reinterpret_cast<const int4*>(p.blocks) + item / p.heads);
  w.h = item % p.heads;
  w.row0 = b.x;
  w.rows = b.y;
  w.pos0 = b.z;
  w.kv0 = b.w;
  w.k_lo = p.first_key(w.pos0);
  w.n_kept = kKeep ? min(p.keep_first, w.k_lo) : 0;
  w.shift = (w.n_kept + 127) / 128;
  w.kept0 = kKeep && p.kept != nullptr ? __ldg(p.kept + item / p.heads) : b.w;
  w.jbA = 0;
  w.jeA = w.shift + (w.pos0 + min(128, w.rows) - 1 - w.k_lo) / 128 + 1;
  w.jbB = w.jeB = 0;
  if (w.rows > 128) {
    // rows that keep first keys walk all tiles: those between the kept ones and their window are masked out
    w.jbB = kKeep && p.keep_first > 0 ? 0 : (p.first_key(w.pos0 + 128) - w.k_lo) / 128;
    w.jeB = w.shift + (w.pos0 + w.rows - 1 - w.k_lo) / 128 + 1;
  }
  w.je = max(w.jeA, w.jeB);
  return true;
}

template <int ND, int NR, int NV, bool kBias>
__global__ void __launch_bounds__(kThreads, 1)
prompt_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_qr,
              const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_kr,
              const __grid_constant__ CUtensorMap tm_v, const Dev p) {
  using C = Cfg<ND, NR, NV, kBias>;
  constexpr int KS = C::kKStages, VS = C::kVStages;
  constexpr bool kKeep = NR == 0;
  extern __shared__ __align__(1024) uint8_t smem[];
  if (smem_u32(smem) & 1023u) {  // the swizzled tiles need a 1 KiB aligned base; uniform early exit
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgument);
    return;
  }
  uint8_t* sQ = smem;                              // [2] query tiles
  uint8_t* sK = sQ + 2 * C::kQBytes;               // [KS]
  uint8_t* sV = sK + KS * C::kKBytes;              // [VS]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + VS * C::kVBytes);
  uint64_t *q_full = bars, *q_empty = bars + 2, *k_full = bars + 4, *k_empty = bars + 6, *v_full = bars + 8, *v_empty = bars + 10,
           *s_full = bars + 12, *p_full = bars + 14, *o_done = bars + 16, *group = bars + 18;      // two each
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 20);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* s_bias = reinterpret_cast<float*>(bars + 32);   // [2][kBiasTable], entry kBiasNear + distance, in units of log2

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int x = 0; x < 2; ++x) {
      mbar_init(&q_full[x], 1);
      mbar_init(&q_empty[x], 1);
      mbar_init(&k_full[x], 1);
      mbar_init(&k_empty[x], 1);
      mbar_init(&v_full[x], 1);
      mbar_init(&v_empty[x], 1);
      mbar_init(&s_full[x], 1);
      mbar_init(&p_full[x], 4);  // one arrival per softmax warp of the group
      mbar_init(&o_done[x], 1);
      mbar_init(&group[x], 4);   // the warps of one softmax group among themselves
    }
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 9) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 8) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      int nq[2] = {0, 0}, n_kv = 0;
      bool ok = true;
      Work w;
      auto wait = [&](uint64_t* bar, int parity) {
        if (mbar_wait_bounded(bar, parity, abort_flag)) return true;
        atomicCAS(p.status, 0, kStatusTimeoutProducer);
        return false;
      };
      for (int round = 0; ok && next_work<kKeep>(p, round, w); ++round) {
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          if (x == 1 && w.jeB <= w.jbB) continue;
          ok = ok && wait(&q_empty[x], (nq[x] & 1) ^ 1);   // the previous item's Q K^T are done
          if (!ok) break;
          ++nq[x];
          mbar_arrive_expect_tx(&q_full[x], C::kQBytes);
          uint8_t* d = sQ + x * C::kQBytes;
#pragma unroll
          for (int s = 0; s < ND; ++s) tma_load_3d(d + s * kSlab, &tm_q, &q_full[x], 64 * s, w.h, w.row0 + x * 128);
          if constexpr (NR > 0) tma_load_3d(d + ND * kSlab, &tm_qr, &q_full[x], 0, w.h, w.row0 + x * 128);
        }
        const int hk = kKeep ? w.h / p.rep : w.h;
        for (int j = 0; ok && j < w.je; ++j, ++n_kv) {
          const int row = (j < w.shift ? w.kept0 : w.kv0) + w.first_key(j);
          const int s = n_kv % KS, v = n_kv % VS;
          ok = wait(&k_empty[s], ((n_kv / KS) & 1) ^ 1);
          if (!ok) break;
          mbar_arrive_expect_tx(&k_full[s], C::kKBytes);
          uint8_t* d = sK + s * C::kKBytes;
#pragma unroll
          for (int c = 0; c < ND; ++c) tma_load_3d(d + c * kSlab, &tm_k, &k_full[s], 64 * c, hk, row);
          if constexpr (NR > 0) tma_load_3d(d + ND * kSlab, &tm_kr, &k_full[s], 0, 0, row);
          ok = wait(&v_empty[v], ((n_kv / VS) & 1) ^ 1);
          if (!ok) break;
          mbar_arrive_expect_tx(&v_full[v], C::kVBytes);
#pragma unroll
          for (int c = 0; c < NV; ++c) tma_load_3d(sV + v * C::kVBytes + c * kSlab, &tm_v, &v_full[v], 64 * c, hk, row);
        }
      }
    }
  } else if (warp == 9) {
    // ------------------------------------------------------------------ MMA issuer: the warp walks, one elected lane issues
    const bool leader = elect_one();
    const uint32_t idesc_s = make_idesc(kFmtBF16, kFmtBF16, false, false, 128, 128);
    const uint32_t idesc_o = make_idesc(kFmtBF16, kFmtBF16, false, true, 128, NV * 64);
    int nq[2] = {0, 0}, np[2] = {0, 0}, n_kv = 0;
    bool ok = true;
    Work w;
    auto wait = [&](uint64_t* bar, int parity) {
      if (__all_sync(0xffffffffu, mbar_wait_bounded(bar, parity, abort_flag))) return true;
      if (leader) atomicCAS(p.status, 0, kStatusTimeoutMma);
      return false;
    };
    for (int round = 0; ok && next_work<kKeep>(p, round, w); ++round) {
      ok = wait(&q_full[0], nq[0] & 1);
      ++nq[0];
      if (ok && w.jeB > w.jbB) {
        ok = wait(&q_full[1], nq[1] & 1);
        ++nq[1];
      }
      const int kv0 = n_kv;
      for (int j = 0; ok && j <= w.je; ++j) {
        const int n = kv0 + j, m = n - 1;          // running numbers of key tiles j and j - 1
        if (j < w.je) ok = wait(&k_full[n % KS], (n / KS) & 1);
        if (ok && j > 0) ok = wait(&v_full[m % VS], (m / VS) & 1);
        if (!ok) break;
        const uint64_t dK = desc_kmajor(smem_u32(sK + (n % KS) * C::kKBytes), 128, 0);
        const uint64_t dV = desc_mnmajor(smem_u32(sV + ((m + VS) % VS) * C::kVBytes), 128, 0);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int jb = x == 0 ? w.jbA : w.jbB, je = x == 0 ? w.jeA : w.jeB;
          const uint32_t tmem_s = tmem_base + x * 128, tmem_o = tmem_base + 256 + x * 128;
          if (ok && j - 1 >= jb && j - 1 < je) {   // P_x(j-1) V(j-1)
            ok = wait(&p_full[x], np[x] & 1);
            if (ok) {
              ++np[x];
              tc_fence_after_sync();
              const uint32_t acc0 = j - 1 > jb ? 1u : 0u;
              if (leader) {
#pragma unroll
                for (int ks = 0; ks < 8; ++ks)
                  umma_f16_ts(tmem_o, tmem_s + ks * 8, dV + kstep_mnmajor(ks), idesc_o, ks > 0 ? 1u : acc0);
                umma_commit(&o_done[x]);
              }
            }
          }
          if (ok && j >= jb && j < je) {           // S_x(j) = Q_x K(j)^T, own part then shared part
            tc_fence_after_sync();
            const uint64_t dQ = desc_kmajor(smem_u32(sQ + x * C::kQBytes), 128, 0);
            if (leader) {
              for (int ks = 0; ks < p.ksteps; ++ks)
                umma_f16_ss(tmem_s, dQ + kstep_kmajor(128, ks), dK + kstep_kmajor(128, ks), idesc_s, ks > 0 ? 1u : 0u);
              for (int ks = ND * 4; NR > 0 && ks < ND * 4 + p.rsteps; ++ks)
                umma_f16_ss(tmem_s, dQ + kstep_kmajor(128, ks), dK + kstep_kmajor(128, ks), idesc_s, 1u);
              umma_commit(&s_full[x]);
              if (j + 1 == je) umma_commit(&q_empty[x]);
            }
          }
        }
        if (ok && leader) {
          if (j < w.je) umma_commit(&k_empty[n % KS]);
          if (j > 0) umma_commit(&v_empty[m % VS]);
        }
        __syncwarp();
      }
      n_kv = kv0 + w.je;
    }
  } else {
    // ------------------------------------------------------------------ softmax + output rows
    const int x = warp >> 2, r = (warp & 3) * 32 + lane;   // query tile of this group; row inside it == TMEM lane
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t tmem_s = tmem_base + x * 128 + lane_addr, tmem_o = tmem_base + 256 + x * 128 + lane_addr;
    const float sc = p.scale * kLog2e;
    int meets = 0;
    int cnt = 0;   // key tiles this group has processed: phase counter of s_full / o_done
    bool ok = true;
    Work w;
    auto wait = [&](uint64_t* bar, int parity) {
      if (__all_sync(0xffffffffu, mbar_wait_bounded(bar, parity, abort_flag))) return true;
      if (lane == 0) atomicCAS(p.status, 0, kStatusTimeoutEpilogue);
      return false;
    };
    auto meet = [&]() {      // barrier of the group's four warps
      __syncwarp();
      if (lane == 0) mbar_arrive(&group[x]);
      return wait(&group[x], meets++ & 1);
    };
    for (int round = 0; ok && next_work<kKeep>(p, round, w); ++round) {
      const int jb = x == 0 ? w.jbA : w.jbB, je = x == 0 ? w.jeA : w.jeB;
      if (je <= jb) continue;
      const int p0 = w.pos0 + x * 128, pos = p0 + r;
      const int row_lo = p.first_key(pos), last_lo = p.first_key(p0 + 127);
      const float* bias = nullptr;
      float b_far = 0.0f;
      if constexpr (kBias) {
        // this head's biases for distances -kBiasNear .. bias_len + kBiasFar - 1, the last one from bias_len on
        float* table = s_bias + x * kBiasTable;
        const float* src = p.bias + static_cast<int64_t>(w.h) * p.bias_len;
        ok = meet();                               // the group has left the previous item's table
        if (!ok) break;
        for (int i = r; i < kBiasNear + p.bias_len + kBiasFar; i += 128)
          table[i] = __ldg(src + min(max(i - kBiasNear, 0), p.bias_len - 1)) * kLog2e;
        b_far = __ldg(src + p.bias_len - 1) * kLog2e;
        ok = meet();
        if (!ok) break;
        bias = table + kBiasNear + pos;
      }
      float m_ref = -INFINITY, l_run = 0.0f;
      for (int j = jb; j < je; ++j, ++cnt) {
        const int k0 = w.first_key(j);
        ok = wait(&s_full[x], cnt & 1);
        if (!ok) break;
        tc_fence_after_sync();
        uint32_t sv[4][32];
#pragma unroll
        for (int cc = 0; cc < 4; ++cc) tmem_ld_32x32b_x32(tmem_s + cc * 32, sv[cc]);
        tmem_ld_wait();
        // scores in units of log2: sc * product + add; a tile that no row is far from gets its biases one by one
        float mul = sc, add = 0.0f;
        if constexpr (kBias) {
          add = b_far;
          if (p0 - k0 - 127 < p.bias_len - 1) {
            mul = 1.0f;
            add = 0.0f;
            const float* b = bias - k0;
#pragma unroll
            for (int cc = 0; cc < 4; ++cc)
#pragma unroll
              for (int c = 0; c < 32; ++c) sv[cc][c] = __float_as_uint(fmaf(__uint_as_float(sv[cc][c]), sc, b[-(cc * 32 + c)]));
          }
        }
        const bool need_mask = (kKeep && j < w.shift) || k0 + 127 > p0 || k0 < last_lo;
        if (need_mask) {
          // column c is visible iff clo <= c <= chi; kept keys: those before k_lo, and in later tiles a row's window or, for a
          // tile that still holds kept keys, everything below keep_first
          int clo = row_lo - k0, chi = pos - k0;
          if (kKeep && j < w.shift) {
            clo = 0;
            chi = min(chi, w.n_kept - 1 - k0);
          } else if (kKeep && k0 < p.keep_first) {
            const int keep = p.keep_first - k0;            // columns below it stay visible
#pragma unroll
            for (int cc = 0; cc < 4; ++cc)
#pragma unroll
              for (int c = 0; c < 32; ++c)
                if (cc * 32 + c >= keep && cc * 32 + c < clo) sv[cc][c] = 0xff800000u;
            clo = 0;
          }
#pragma unroll
          for (int cc = 0; cc < 4; ++cc)
#pragma unroll
            for (int c = 0; c < 32; ++c)
              if (cc * 32 + c < clo || cc * 32 + c > chi) sv[cc][c] = 0xff800000u;  // -inf
        }
        float m0 = -INFINITY, m1 = -INFINITY, m2 = -INFINITY, m3 = -INFINITY;
#pragma unroll
        for (int cc = 0; cc < 4; ++cc)
#pragma unroll
          for (int c = 0; c < 32; c += 4) {
            m0 = fmaxf(m0, __uint_as_float(sv[cc][c]));
            m1 = fmaxf(m1, __uint_as_float(sv[cc][c + 1]));
            m2 = fmaxf(m2, __uint_as_float(sv[cc][c + 2]));
            m3 = fmaxf(m3, __uint_as_float(sv[cc][c + 3]));
          }
        const float m_new = fmaxf(m_ref, fmaf(fmaxf(fmaxf(m0, m1), fmaxf(m2, m3)), mul, add));
        const bool grow = m_new - kRescaleStep > m_ref;
        if (__any_sync(0xffffffffu, grow)) {
          const float alpha = grow ? ex2f(m_ref - m_new) : 1.0f;  // m_ref == -inf -> 0
          if (grow) {
            l_run *= alpha;
            m_ref = m_new;
          }
          if (j > jb) {  // the output tile holds the sums of the earlier key tiles
            ok = wait(&o_done[x], (cnt - 1) & 1);
            if (!ok) break;
            tc_fence_after_sync();
#pragma unroll
            for (int cc = 0; cc < NV * 2; ++cc) {
              uint32_t ov[32];
              tmem_ld_32x32b_x32(tmem_o + cc * 32, ov);
              tmem_ld_wait();
#pragma unroll
              for (int c = 0; c < 32; ++c) ov[c] = __float_as_uint(__uint_as_float(ov[c]) * alpha);
              tmem_st_32x32b_x32(tmem_o + cc * 32, ov);
            }
            tmem_st_wait();
          }
        }
        const float m_use = (m_ref == -INFINITY ? 0.0f : m_ref) - add;
        float r0 = 0.0f, r1 = 0.0f, r2 = 0.0f, r3 = 0.0f;
#pragma unroll
        for (int cc = 0; cc < 4; ++cc) {
          uint32_t pk[16];
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            float e[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) e[i] = ex2f(fmaf(__uint_as_float(sv[cc][8 * g + i]), mul, -m_use));  // -inf -> 0
            r0 += e[0] + e[4];
            r1 += e[1] + e[5];
            r2 += e[2] + e[6];
            r3 += e[3] + e[7];
            pk[4 * g + 0] = pack_bf16x2(e[0], e[1]);
            pk[4 * g + 1] = pack_bf16x2(e[2], e[3]);
            pk[4 * g + 2] = pack_bf16x2(e[4], e[5]);
            pk[4 * g + 3] = pack_bf16x2(e[6], e[7]);
          }
          tmem_st_32x32b_x16(tmem_s + cc * 16, pk);  // two probabilities per column
        }
        l_run += (r0 + r1) + (r2 + r3);
        tmem_st_wait();
        tc_fence_before_sync();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_full[x]);
      }
      if (!ok) break;
      ok = wait(&o_done[x], (cnt - 1) & 1);        // the last P V has retired
      if (!ok) break;
      tc_fence_after_sync();
      const bool row_ok = x * 128 + r < w.rows;
      const int64_t row = w.row0 + x * 128 + r;
      if (kKeep && p.sink != nullptr) l_run += ex2f(p.sink[w.h] * kLog2e - m_ref);
      const float inv = row_ok ? (p.gate != nullptr ? p.gate[row * p.heads + w.h] : 1.0f) / l_run : 0.0f;
      __nv_bfloat16* orow = p.out + row * p.ldo + static_cast<int64_t>(w.h) * p.vdim;
#pragma unroll
      for (int cc = 0; cc < NV * 2; ++cc) {
        uint32_t ov[32];
        tmem_ld_32x32b_x32(tmem_o + cc * 32, ov);
        tmem_ld_wait();
        if (!row_ok) continue;
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          if (cc * 32 + g * 8 >= p.vdim) continue;
          uint4 wv;
          wv.x = pack_bf16x2(__uint_as_float(ov[8 * g + 0]) * inv, __uint_as_float(ov[8 * g + 1]) * inv);
          wv.y = pack_bf16x2(__uint_as_float(ov[8 * g + 2]) * inv, __uint_as_float(ov[8 * g + 3]) * inv);
          wv.z = pack_bf16x2(__uint_as_float(ov[8 * g + 4]) * inv, __uint_as_float(ov[8 * g + 5]) * inv);
          wv.w = pack_bf16x2(__uint_as_float(ov[8 * g + 6]) * inv, __uint_as_float(ov[8 * g + 7]) * inv);
          *reinterpret_cast<uint4*>(orow + cc * 32 + g * 8) = wv;
        }
      }
      tc_fence_before_sync();
    }
  }

  tc_fence_before_sync();
  __syncthreads();
  if (*abort_flag != 0) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(2000);
    __syncthreads();
  }
  if (warp == 9) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, 512);
  }
}

// tensor map of [rows][heads][columns], box 128 x 1 x 64: columns past a part's width arrive as zeros
int part_map(CUtensorMap* m, const void* base, int cols, int heads, int rows, int64_t head_ld, int64_t row_ld) {
  nx::EncodeTiledFn fn = nx::encode_tiled_fn();
  if (fn == nullptr) return -3;
  cuuint64_t dims[3] = {static_cast<cuuint64_t>(cols), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(rows)};
  cuuint64_t strides[2] = {static_cast<cuuint64_t>(head_ld) * 2, static_cast<cuuint64_t>(row_ld) * 2};
  cuuint32_t box[3] = {64, 1, 128}, one[3] = {1, 1, 1};
  return fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, one, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS
             ? 0
             : -4;
}

struct Maps {
  CUtensorMap q, qr, k, kr, v;
};

template <int ND, int NR, int NV, bool kBias>
int launch(const Maps& t, const Dev& p, cudaStream_t st) {
  constexpr int kSmem = Cfg<ND, NR, NV, kBias>::kSmem;
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(prompt_kernel<ND, NR, NV, kBias>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem) != cudaSuccess) return -2;
    once = true;
  }
  int sms = 0, dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) return -2;
  prompt_kernel<ND, NR, NV, kBias><<<std::min(p.items, sms), kThreads, kSmem, st>>>(t.q, t.qr, t.k, t.kr, t.v, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
template <int NR, bool kBias>
int launch_sizes(int dim, int vdim, const Maps& t, const Dev& p, cudaStream_t st) {
  if (dim <= 64) return vdim <= 64 ? launch<1, NR, 1, kBias>(t, p, st) : launch<1, NR, 2, kBias>(t, p, st);
  return vdim <= 64 ? launch<2, NR, 1, kBias>(t, p, st) : launch<2, NR, 2, kBias>(t, p, st);
}

// copies the cache rows of a segment list into one packed buffer: keys `base` .. of every segment, 16 bytes per thread
__global__ void latent_gather_kernel(const uint4* __restrict__ cache, uint4* __restrict__ dst, const int32_t* __restrict__ table,
                                     const int32_t* __restrict__ list, int n, int max_blocks, int block_size, int chunks) {
  // list [n][4]: first destination row, rows, first position, sequence
  const int seg = blockIdx.y, count = list[seg * 4 + 1];
  const int64_t d0 = list[seg * 4], seq = list[seg * 4 + 3];
  const int p0 = list[seg * 4 + 2];
  for (int64_t i = blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x; i < static_cast<int64_t>(count) * chunks;
       i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int k = static_cast<int>(i / chunks), c = static_cast<int>(i % chunks), j = p0 + k;
    const int64_t slot = static_cast<int64_t>(table[seq * max_blocks + j / block_size]) * block_size + j % block_size;
    dst[(d0 + k) * chunks + c] = cache[slot * chunks + c];
  }
}

}  // namespace

extern "C" int nx_latent_gather(const void* cache, void* dst, const int32_t* block_table, const int32_t* list, int segments,
                                int longest, int max_blocks, int block_size, int row, nx_stream_t stream) {
  if (segments < 0 || segments > 65535 || block_size <= 0 || max_blocks <= 0 || row <= 0 || (row & 7)) return -1;
  if ((reinterpret_cast<uintptr_t>(cache) & 15) || (reinterpret_cast<uintptr_t>(dst) & 15)) return -1;
  if (segments == 0 || longest <= 0) return 0;
  const int64_t work = (static_cast<int64_t>(longest) * (row / 8) + 255) / 256;
  const dim3 grid(static_cast<unsigned>(std::min<int64_t>(work, 1024)), segments);
  latent_gather_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const uint4*>(cache), static_cast<uint4*>(dst), block_table, list, segments, max_blocks, block_size, row / 8);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

extern "C" int nx_latent_prompt(const NxLatentPromptArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->status == nullptr || a->blocks == nullptr || a->heads <= 0 || !(a->scale > 0.0f)) return -1;
  if (a->dim <= 0 || a->dim > 128 || a->rot <= 0 || a->rot > 64 || a->vdim <= 0 || a->vdim > 128) return -1;
  if ((a->dim & 15) || (a->rot & 15) || (a->vdim & 7)) return -1;
  if ((a->ldq | a->ldkv | a->ld_lat | a->ldo | a->q_head) & 7) return -1;
  for (const void* ptr : {a->q, a->kv, a->lat, static_cast<const void*>(a->out)})
    if (ptr == nullptr || (reinterpret_cast<uintptr_t>(ptr) & 15)) return -1;
  if (a->n_blocks <= 0) return 0;
  const auto* q = static_cast<const __nv_bfloat16*>(a->q);
  const auto* kv = static_cast<const __nv_bfloat16*>(a->kv);
  const auto* lat = static_cast<const __nv_bfloat16*>(a->lat);
  const int H = a->heads;
  Maps t;
  int rc;
  if ((rc = part_map(&t.q, q, a->dim, H, a->q_rows, a->q_head, a->ldq))) return rc;
  if ((rc = part_map(&t.qr, q + a->dim, a->rot, H, a->q_rows, a->q_head, a->ldq))) return rc;
  if ((rc = part_map(&t.k, kv, a->dim, H, a->kv_rows, a->dim, a->ldkv))) return rc;
  if ((rc = part_map(&t.v, kv + static_cast<int64_t>(H) * a->dim, a->vdim, H, a->kv_rows, a->vdim, a->ldkv))) return rc;
  if ((rc = part_map(&t.kr, lat + a->rank, a->rot, 1, a->kv_rows, a->ld_lat, a->ld_lat))) return rc;
  Dev p{};
  p.blocks = a->blocks;
  p.out = static_cast<__nv_bfloat16*>(a->out);
  p.gate = a->gate;
  p.status = a->status;
  p.ldo = a->ldo;
  p.items = a->n_blocks * H;
  p.heads = H;
  p.rep = 1;
  p.vdim = a->vdim;
  p.window = a->window;
  p.ksteps = a->dim / 16;
  p.rsteps = a->rot / 16;
  p.scale = a->scale;
  return launch_sizes<1, false>(a->dim, a->vdim, t, p, static_cast<cudaStream_t>(stream));
}

extern "C" int nx_window_prompt(const NxWindowPromptArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->status == nullptr || a->blocks == nullptr || a->heads <= 0 || a->kv_heads <= 0 || !(a->scale > 0.0f)) return -1;
  if (a->heads % a->kv_heads || a->keep_first < 0 || a->chunk < 0) return -1;
  if (a->bias != nullptr && (a->bias_len <= 0 || a->bias_len > kBiasMax)) return -1;
  if (a->dim <= 0 || a->dim > 128 || (a->dim & 15) || a->vdim <= 0 || a->vdim > 128 || (a->vdim & 7)) return -1;
  if ((a->ldq | a->ldk | a->ldv | a->ldo) & 7) return -1;
  for (const void* ptr : {a->q, a->k, a->v, static_cast<const void*>(a->out), static_cast<const void*>(a->blocks)})
    if (ptr == nullptr || (reinterpret_cast<uintptr_t>(ptr) & 15)) return -1;
  if (a->n_blocks <= 0) return 0;
  Maps t;
  int rc;
  if ((rc = part_map(&t.q, a->q, a->dim, a->heads, a->q_rows, a->dim, a->ldq))) return rc;
  if ((rc = part_map(&t.k, a->k, a->dim, a->kv_heads, a->kv_rows, a->dim, a->ldk))) return rc;
  if ((rc = part_map(&t.v, a->v, a->vdim, a->kv_heads, a->kv_rows, a->vdim, a->ldv))) return rc;
  t.qr = t.q;                // not used without a shared key part
  t.kr = t.k;
  Dev p{};
  p.blocks = a->blocks;
  p.kept = a->kept;
  p.out = static_cast<__nv_bfloat16*>(a->out);
  p.sink = a->sink;
  p.gate = a->gate;
  p.bias = a->bias;
  p.bias_len = a->bias_len;
  p.chunk = a->chunk;
  p.status = a->status;
  p.ldo = a->ldo;
  p.items = a->n_blocks * a->heads;
  p.heads = a->heads;
  p.rep = a->heads / a->kv_heads;
  p.vdim = a->vdim;
  p.window = a->window;
  p.keep_first = a->window > 0 || a->chunk > 0 ? a->keep_first : 0;
  p.ksteps = a->dim / 16;
  p.scale = a->scale;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return p.bias != nullptr ? launch_sizes<0, true>(a->dim, a->vdim, t, p, st) : launch_sizes<0, false>(a->dim, a->vdim, t, p, st);
}
