// Attention of prompt segments on tcgen05 where every query head's weights meet the values of every KV head: heads that mix their
// weights (see nx_api_mixers.h).  out_h = sum_g talk[h][g] (P_g V of the KV head of h), so the kernel forms P_g V_c for all g and c and
// nx_head_mix takes the mixture.
//
// A work item is a tile of 128 query rows, one query head and up to 256 columns of values (several KV heads side by side): the scores and
// the softmax are formed once for all of them.  Key tiles have 64 keys; S lives four times in TMEM (columns 0-255), O behind it
// (256-511).  One persistent CTA per SM: two softmax groups of four warps take the key tiles of the CTA's running count in turn; one warp
// issues the products Q K^T up to four tiles ahead, another P V.  Both groups add to one O, so they share the row maxima that O is scaled
// by: tile j passes them on to tile j + 1, between the two warps that own the same 32 rows.  O is rescaled only when a row's maximum has
// grown by 2^8.  A head's table of biases (in units of log2, extended to both sides) arrives by bulk copy beside its queries.
#include "flash_common.cuh"
#include "nx_api_mixers.h"
#include "sm100_ptx.cuh"
#include "tensor_map.h"

#include <algorithm>

namespace {
using namespace nx;

constexpr int kGroups = 2;           // softmax groups
constexpr int kThreads = (kGroups * 4 + 3) * 32;   // after the softmax warps: TMA, Q K^T, P V
constexpr int kKeys = 64;            // keys of a tile
constexpr int kTilesAhead = 4;       // score tiles in TMEM
constexpr int kSlab = 128 * 128;     // bytes of [128 rows][64 columns]
constexpr int kKeySlab = kKeys * 128;  // of [64 keys][64 columns]
constexpr int kSlabs = 4;            // 64-column slabs of values in one item
constexpr int kBiasNear = NX_TALK_BIAS_NEAR, kBiasTable = NX_TALK_BIAS_NEAR + NX_TALK_BIAS_MAX + NX_TALK_BIAS_FAR;

// ND: 64-column slabs of a key
template <int ND>
struct Cfg {
  static constexpr int kQStages = ND == 1 ? 2 : 1, kKStages = 4, kVStages = ND == 1 ? 4 : 3;
  static constexpr int kQBytes = ND * kSlab, kKBytes = ND * kKeySlab, kVBytes = kSlabs * kKeySlab;
  static constexpr int kTiles = kQStages * kQBytes + kKStages * kKBytes + kVStages * kVBytes;
  static constexpr int kBarriers = 512, kStats = 128 * 4 + kGroups * 128 * 8;
  static constexpr int kSmem = kTiles + kBarriers + kStats + 2 * kBiasTable * 4;
  static_assert(kSmem <= 227 * 1024, "shared memory");
};

struct Dev {
  const int32_t* blocks;     // [n_blocks][4]: first row, rows, position of the first row, buffer row of position 0
  const float* bias;         // [heads][bias_pitch], null: none
  __nv_bfloat16* out;
  int* status;
  int64_t ldo;
  int items, heads, kv_heads, rep, vdim, window, chunk, bias_len, bias_pitch;
  int slabs, at_once, passes;   // slabs of one KV head's values (1, 2), KV heads of one item, items per (tile, head)
  int wide_store;               // output rows and heads start on 32 bytes
  float scale;
  __device__ __forceinline__ int first_key(int pos) const {
    const int lo = window > 0 ? max(0, pos - window + 1) : 0;
    return chunk > 0 ? max(lo, pos / chunk * chunk) : lo;
  }
};

// 32 bytes, 32-byte aligned
__device__ __forceinline__ void store32(void* p, const uint32_t* v) {
  asm volatile("st.global.v8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(p), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]),
               "r"(v[5]), "r"(v[6]), "r"(v[7])
               : "memory");
}

struct Work {
  int h, hk, c0;                   // query head, its KV head, first KV head of the values
  int row0, rows, pos0, kv0, k_lo, n;   // n: key tiles
};
// the CTA's items in order; an item whose half block holds no rows is left out by every role
__device__ __forceinline__ bool next_work(const Dev& p, int& round, Work& w) {
  const int G = static_cast<int>(gridDim.x), c = static_cast<int>(blockIdx.x);
  for (;; ++round) {
    const int item = round * G + ((round & 1) ? (G - 1 - c) : c);
    if (round * G >= p.items) return false;
    if (item >= p.items) continue;
    const int per = 2 * p.heads * p.passes, block = item / per, sub = item % per;
    const int4 b = __ldg(reinterpret_cast<const int4*>(p.blocks) + block);
    const int half = 1 - sub / (p.heads * p.passes);       // the half with more keys first
    w.rows = min(128, b.y - half * 128);
    if (w.rows <= 0) continue;
    w.h = sub % p.heads;
    w.hk = w.h / p.rep;
    w.c0 = sub / p.heads % p.passes * p.at_once;
    w.row0 = b.x + half * 128;
    w.pos0 = b.z + half * 128;
    w.kv0 = b.w;
    w.k_lo = p.first_key(w.pos0);
    w.n = (w.pos0 + w.rows - 1 - w.k_lo) / kKeys + 1;
    ++round;
    return true;
  }
}

template <int ND>
__global__ void __launch_bounds__(kThreads, 1)
talk_prompt_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                   const __grid_constant__ CUtensorMap tm_v, const Dev p) {
  using C = Cfg<ND>;
  constexpr int QS = C::kQStages, KS = C::kKStages, VS = C::kVStages;
  extern __shared__ __align__(1024) uint8_t smem[];
  if (smem_u32(smem) & 1023u) {  // the swizzled tiles need a 1 KiB aligned base; uniform early exit
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadArgument);
    return;
  }
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + QS * C::kQBytes;
  uint8_t* sV = sK + KS * C::kKBytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + C::kTiles);
  uint64_t *q_full = bars, *q_empty = bars + 2, *b_full = bars + 4, *b_empty = bars + 6, *k_full = bars + 8, *k_empty = bars + 12,
           *v_full = bars + 16, *v_empty = bars + 20, *s_full = bars + 24, *p_full = bars + 28, *o_done = bars + 32 /* one per score tile */,
           *chain = bars + 36 /* [groups][4] */, *fin = bars + 52 /* [4] */, *o_free = bars + 56;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 57);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* s_m = reinterpret_cast<float*>(smem + C::kTiles + C::kBarriers);      // [128] row maximum that O is scaled by
  float2* s_l = reinterpret_cast<float2*>(s_m + 128);                          // [groups][128] sum and its maximum
  float* s_bias = reinterpret_cast<float*>(s_l + kGroups * 128);               // [2][kBiasTable]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int x = 0; x < 2; ++x) {
      mbar_init(&q_full[x], 1);
      mbar_init(&q_empty[x], 1);
      mbar_init(&b_full[x], 1);
      mbar_init(&b_empty[x], kGroups * 4);   // one arrival per softmax warp
    }
    for (int x = 0; x < 4; ++x) {
      mbar_init(&k_full[x], 1);
      mbar_init(&k_empty[x], 1);
      mbar_init(&s_full[x], 1);
      mbar_init(&p_full[x], 4);   // one arrival per softmax warp of the group
      mbar_init(&o_done[x], 1);
      mbar_init(&v_full[x], 1);
      mbar_init(&v_empty[x], 1);
    }
    for (int x = 0; x < kGroups * 4; ++x) mbar_init(&chain[x], 1);
    for (int x = 0; x < 4; ++x) mbar_init(&fin[x], kGroups);
    mbar_init(o_free, kGroups * 4);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == kGroups * 4 + 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;

  if (warp >= kGroups * 4) {
    if (warp == kGroups * 4) {
      // ---------------------------------------------------------------- TMA producer
      if (lane == 0) {
        int items = 0, nk = 0, nv = 0, round = 0;
        const int v_bytes = p.at_once * p.slabs * kKeySlab;
        bool ok = true;
        Work w;
        auto wait = [&](uint64_t* bar, int parity) {
          if (mbar_wait_bounded(bar, parity, abort_flag)) return true;
          atomicCAS(p.status, 0, kStatusTimeoutProducer);
          return false;
        };
        auto keys = [&](int j) {
          const int s = nk % KS;
          if (!wait(&k_empty[s], ((nk / KS) & 1) ^ 1)) return false;
          ++nk;
          mbar_arrive_expect_tx(&k_full[s], C::kKBytes);
#pragma unroll
          for (int c = 0; c < ND; ++c)
            tma_load_3d(sK + s * C::kKBytes + c * kKeySlab, &tm_k, &k_full[s], 64 * c, w.hk, w.kv0 + w.k_lo + j * kKeys);
          return true;
        };
        for (; ok && next_work(p, round, w); ++items) {
          const int qs = items % QS;
          ok = wait(&q_empty[qs], ((items / QS) & 1) ^ 1);   // the Q K^T of the item that used it are done
          if (!ok) break;
          mbar_arrive_expect_tx(&q_full[qs], C::kQBytes);
#pragma unroll
          for (int c = 0; c < ND; ++c) tma_load_3d(sQ + qs * C::kQBytes + c * kSlab, &tm_q, &q_full[qs], 64 * c, w.h, w.row0);
          if (p.bias != nullptr) {
            const int b = items & 1;
            ok = wait(&b_empty[b], ((items >> 1) & 1) ^ 1);
            if (!ok) break;
            mbar_arrive_expect_tx(&b_full[b], p.bias_pitch * 4);
            bulk_load(s_bias + b * kBiasTable, p.bias + static_cast<int64_t>(w.h) * p.bias_pitch, p.bias_pitch * 4, &b_full[b]);
          }
          for (int j = 0; ok && j < min(KS, w.n); ++j) ok = keys(j);
          for (int j = 0; ok && j < w.n; ++j, ++nv) {
            const int s = nv % VS;
            ok = wait(&v_empty[s], ((nv / VS) & 1) ^ 1);
            if (!ok) break;
            mbar_arrive_expect_tx(&v_full[s], v_bytes);
            uint8_t* d = sV + s * C::kVBytes;                // one slab of every KV head, then their second slabs
            const int row = w.kv0 + w.k_lo + j * kKeys;
            tma_load_3d(d, &tm_v, &v_full[s], 0, row, w.c0);
            if (p.slabs > 1) tma_load_3d(d + p.at_once * kKeySlab, &tm_v, &v_full[s], 64, row, w.c0);
            if (j + KS < w.n) ok = keys(j + KS);
          }
        }
      }
    } else {
      // ---------------------------------------------------------------- MMA issuers: one lane each
      if (elect_one()) {
        int items = 0, round = 0;
        uint32_t t = 0, ring = 0, ring_phase = 0;      // running number of the key tile; its stage of keys or values
        bool ok = true;
        Work w;
        auto wait = [&](uint64_t* bar, uint32_t parity) {
          if (mbar_try_wait(bar, parity) || mbar_wait_bounded(bar, parity, abort_flag)) return true;
          atomicCAS(p.status, 0, kStatusTimeoutMma);
          return false;
        };
        if (warp == kGroups * 4 + 1) {                 // S(t) = Q K(t)^T
          constexpr uint32_t idesc = make_idesc(kFmtBF16, kFmtBF16, false, false, 128, kKeys);
          const uint64_t dK0 = desc_kmajor(smem_u32(sK), kKeys, 0);
          for (; ok && next_work(p, round, w); ++items) {
            const uint64_t dQ = desc_kmajor(smem_u32(sQ + (items % QS) * C::kQBytes), 128, 0);
            ok = wait(&q_full[items % QS], (items / QS) & 1);
            for (int j = 0; ok && j < w.n; ++j, ++t) {
              const uint32_t b = t % kTilesAhead;
              ok = wait(&o_done[b], ((t / kTilesAhead) & 1) ^ 1) &&    // the weights in these columns have been used
                   wait(&k_full[ring], ring_phase);
              if (!ok) break;
              tc_fence_after_sync();
              const uint64_t dK = dK0 + ring * (C::kKBytes >> 4);
#pragma unroll
              for (int ks = 0; ks < ND * 4; ++ks)      // columns past the head size are zeros
                umma_f16_ss(tmem_base + b * kKeys, dQ + kstep_kmajor(128, ks), dK + kstep_kmajor(kKeys, ks), idesc, ks > 0 ? 1u : 0u);
              umma_commit(&s_full[b]);
              umma_commit(&k_empty[ring]);
              if (j + 1 == w.n) umma_commit(&q_empty[items % QS]);
              if (++ring == KS) {
                ring = 0;
                ring_phase ^= 1;
              }
            }
          }
        } else {                                       // O (+)= P(t) V(t)
          const uint32_t idesc = make_idesc(kFmtBF16, kFmtBF16, false, true, 128, p.at_once * p.slabs * 64);
          const uint64_t dV0 = desc_mnmajor(smem_u32(sV), kKeys, 0);
          for (; ok && next_work(p, round, w); ++items) {
            for (int j = 0; ok && j < w.n; ++j, ++t) {
              const uint32_t b = t % kTilesAhead;
              ok = wait(&v_full[ring], ring_phase) &&
                   (j > 0 || items == 0 || wait(o_free, (items - 1) & 1)) &&      // the rows of the previous item have been read
                   wait(&p_full[b], (t / kTilesAhead) & 1);
              if (!ok) break;
              tc_fence_after_sync();
              const uint64_t dV = dV0 + ring * (C::kVBytes >> 4);
#pragma unroll
              for (int ks = 0; ks < kKeys / 16; ++ks)
                umma_f16_ts(tmem_base + 256, tmem_base + b * kKeys + ks * 8, dV + kstep_mnmajor(ks), idesc, j > 0 || ks > 0 ? 1u : 0u);
              umma_commit(&o_done[b]);
              umma_commit(&v_empty[ring]);
              if (++ring == VS) {
                ring = 0;
                ring_phase ^= 1;
              }
            }
          }
        }
      }
      __syncwarp();
    }
  } else {
    // ------------------------------------------------------------------ softmax + output rows
    const int x = warp >> 2, quad = warp & 3, r = quad * 32 + lane;    // group; row inside the tile == TMEM lane
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t tmem_o = tmem_base + 256 + lane_addr;
    uint64_t *mine = chain + x * 4 + quad, *theirs = chain + ((x + kGroups - 1) % kGroups) * 4 + quad;
    const float sc = p.scale * kLog2e;
    int items = 0, t0 = 0, round = 0;
    bool ok = true;
    Work w;
    auto wait = [&](uint64_t* bar, int parity) {
      if (__all_sync(0xffffffffu, mbar_wait_bounded(bar, parity, abort_flag))) return true;
      if (lane == 0) atomicCAS(p.status, 0, kStatusTimeoutEpilogue);
      return false;
    };
    for (; ok && next_work(p, round, w); ++items) {
      const int pos = w.pos0 + r, row_lo = p.first_key(pos), last_lo = p.first_key(w.pos0 + 127);
      const float* bias = nullptr;
      float b_far = 0.0f;
      if (p.bias != nullptr) {
        ok = wait(&b_full[items & 1], (items >> 1) & 1);
        if (!ok) break;
        bias = s_bias + (items & 1) * kBiasTable + kBiasNear;
        b_far = bias[p.bias_len - 1];
        bias += pos;
      }
      float m_own = -INFINITY, l_run = 0.0f;
      for (int j = (x + kGroups - t0 % kGroups) % kGroups; j < w.n; j += kGroups) {
        const int t = t0 + j, b = t % kTilesAhead, k0 = w.k_lo + j * kKeys;
        const uint32_t tmem_s = tmem_base + b * kKeys + lane_addr;
        ok = wait(&s_full[b], (t / kTilesAhead) & 1);
        if (!ok) break;
        tc_fence_after_sync();
        uint32_t sv[2][32];
        tmem_ld_32x32b_x32(tmem_s, sv[0]);
        tmem_ld_32x32b_x32(tmem_s + 32, sv[1]);
        tmem_ld_wait();
        // Scores in units of log2: mul * product + add; in a tile that has masked columns, or biases of its own for every distance, both
        // are applied at once.
        const bool near = bias != nullptr && w.pos0 - k0 - (kKeys - 1) < p.bias_len - 1;
        const bool masked = k0 + kKeys - 1 > w.pos0 || k0 < last_lo, special = near || masked;
        const float mul = special ? 1.0f : sc, add = special ? 0.0f : b_far;
        if (near) {
          const float* at = bias - k0;
#pragma unroll
          for (int c = 0; c < kKeys; ++c) sv[c >> 5][c & 31] = __float_as_uint(fmaf(__uint_as_float(sv[c >> 5][c & 31]), sc, at[-c]));
        } else if (special) {
#pragma unroll
          for (int c = 0; c < kKeys; ++c) sv[c >> 5][c & 31] = __float_as_uint(fmaf(__uint_as_float(sv[c >> 5][c & 31]), sc, b_far));
        }
        if (masked) {
          const int clo = row_lo - k0, chi = pos - k0;       // column c is visible iff clo <= c <= chi
#pragma unroll
          for (int c = 0; c < kKeys; ++c)
            if (c < clo || c > chi) sv[c >> 5][c & 31] = 0xff800000u;  // -inf
        }
        float m0 = -INFINITY, m1 = -INFINITY, m2 = -INFINITY, m3 = -INFINITY;
#pragma unroll
        for (int c = 0; c < kKeys; c += 4) {
          m0 = fmaxf(m0, __uint_as_float(sv[c >> 5][c & 31]));
          m1 = fmaxf(m1, __uint_as_float(sv[c >> 5][(c & 31) + 1]));
          m2 = fmaxf(m2, __uint_as_float(sv[c >> 5][(c & 31) + 2]));
          m3 = fmaxf(m3, __uint_as_float(sv[c >> 5][(c & 31) + 3]));
        }
        const float m_tile = fmaf(fmaxf(fmaxf(m0, m1), fmaxf(m2, m3)), mul, add);
        // the maxima after tile j - 1, from the warp that has the same rows there
        if (t > 0) {
          ok = wait(theirs, ((t - 1) / kGroups) & 1);
          if (!ok) break;
        }
        const float m_prev = j > 0 ? s_m[r] : -INFINITY;
        const float m_new = fmaxf(m_prev, m_tile);
        const bool grow = m_new - kRescaleStep > m_prev;
        const float m_ref = grow ? m_new : m_prev;
        s_m[r] = m_ref;
        __syncwarp();
        if (lane == 0) mbar_arrive(mine);
        if (j > 0 && __any_sync(0xffffffffu, grow)) {   // the output tile holds the sums of the earlier key tiles
          const float alpha = grow ? ex2f(m_prev - m_new) : 1.0f;
          ok = wait(&o_done[(t - 1) % kTilesAhead], ((t - 1) / kTilesAhead) & 1);   // S(t) came after P(t - 4) V, so this phase is next
          if (!ok) break;
          tc_fence_after_sync();
#pragma unroll 1
          for (int cc = 0; cc < p.at_once * p.slabs * 2; ++cc) {
            uint32_t ov[32];
            tmem_ld_32x32b_x32(tmem_o + cc * 32, ov);
            tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < 32; ++c) ov[c] = __float_as_uint(__uint_as_float(ov[c]) * alpha);
            tmem_st_32x32b_x32(tmem_o + cc * 32, ov);
          }
          tmem_st_wait();
        }
        if (m_ref != m_own) {
          l_run *= ex2f(m_own - m_ref);               // m_own == -inf -> 0
          m_own = m_ref;
        }
        const float m_use = (m_ref == -INFINITY ? 0.0f : m_ref) - add;
        float r0 = 0.0f, r1 = 0.0f, r2 = 0.0f, r3 = 0.0f;
#pragma unroll
        for (int cc = 0; cc < 2; ++cc) {
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
        if (lane == 0) mbar_arrive(&p_full[b]);
      }
      if (!ok) break;
      // the groups' sums, each relative to the maximum it last saw; not before all warps are done with the previous item's
      if (items > 0) {
        ok = wait(o_free, (items - 1) & 1);
        if (!ok) break;
      }
      s_l[x * 128 + r] = make_float2(l_run, m_own);
      __syncwarp();
      if (lane == 0) {
        if (p.bias != nullptr) mbar_arrive(&b_empty[items & 1]);
        mbar_arrive(&fin[quad]);
      }
      ok = wait(&fin[quad], items & 1);
      if (!ok) break;
      float m_end = -INFINITY, total = 0.0f;
#pragma unroll
      for (int g = 0; g < kGroups; ++g) m_end = fmaxf(m_end, s_l[g * 128 + r].y);
#pragma unroll
      for (int g = 0; g < kGroups; ++g) {
        const float2 part = s_l[g * 128 + r];
        total += part.y == -INFINITY ? 0.0f : part.x * ex2f(part.y - m_end);
      }
      const int t_last = t0 + w.n - 1;
      // the last P V has retired; S(t_last), which a group has seen, came after P(t_last - 4) V
      ok = wait(&o_done[t_last % kTilesAhead], (t_last / kTilesAhead) & 1);
      if (!ok) break;
      tc_fence_after_sync();
      const bool row_ok = r < w.rows;
      const float inv = row_ok ? 1.0f / total : 0.0f;
      __nv_bfloat16* orow = p.out + static_cast<int64_t>(w.row0 + r) * p.ldo + (static_cast<int64_t>(w.h) * p.kv_heads + w.c0) * p.vdim;
      const int heads_here = min(p.at_once, p.kv_heads - w.c0);
#pragma unroll 1
      for (int cc = x; cc < p.at_once * p.slabs * 2; cc += kGroups) {      // 32 columns each, the groups in turn
        const int s = cc >> 1, second = s >= p.at_once ? 1 : 0, c = s - second * p.at_once, d0 = second * 64 + (cc & 1) * 32;
        uint32_t ov[32];
        tmem_ld_32x32b_x32(tmem_o + cc * 32, ov);
        tmem_ld_wait();
        if (row_ok && c < heads_here && d0 < p.vdim) {
          uint32_t pk[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) pk[i] = pack_bf16x2(__uint_as_float(ov[2 * i]) * inv, __uint_as_float(ov[2 * i + 1]) * inv);
          __nv_bfloat16* o = orow + static_cast<int64_t>(c) * p.vdim + d0;
          if (p.wide_store && d0 + 32 <= p.vdim) {       // whole sectors
            store32(o, pk);
            store32(o + 16, pk + 8);
          } else {
#pragma unroll
            for (int g = 0; g < 4; ++g)
              if (d0 + g * 8 < p.vdim) *reinterpret_cast<uint4*>(o + g * 8) = make_uint4(pk[4 * g], pk[4 * g + 1], pk[4 * g + 2], pk[4 * g + 3]);
          }
        }
        __syncwarp();
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(o_free);
      t0 += w.n;
    }
  }

  tc_fence_before_sync();
  __syncthreads();
  if (*abort_flag != 0) {       // copies in flight still write to this CTA's shared memory
    const uint64_t t_end = globaltimer_ns();
    while (globaltimer_ns() - t_end < 2000000ull) __nanosleep(2000);
    __syncthreads();
  }
  if (warp == kGroups * 4 + 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, 512);
  }
}

// Tensor map of [rows][heads][columns]: columns past a head's width and heads past the last arrive as zeros.  box_heads 0: box of
// box_rows rows of one head, coordinates (column, head, row); else of box_heads slabs of box_rows rows, coordinates (column, row, head).
int head_map(CUtensorMap* m, const void* base, int cols, int heads, int rows, int64_t row_ld, int box_rows, int box_heads) {
  nx::EncodeTiledFn fn = nx::encode_tiled_fn();
  if (fn == nullptr) return -3;
  const int head = box_heads > 0 ? 2 : 1, row = 3 - head;
  cuuint64_t dims[3] = {static_cast<cuuint64_t>(cols), 0, 0}, strides[2];
  cuuint32_t box[3] = {64, 1, 1}, one[3] = {1, 1, 1};
  dims[head] = static_cast<cuuint64_t>(heads);
  dims[row] = static_cast<cuuint64_t>(rows);
  strides[head - 1] = static_cast<cuuint64_t>(cols) * 2;
  strides[row - 1] = static_cast<cuuint64_t>(row_ld) * 2;
  box[head] = static_cast<cuuint32_t>(std::max(1, box_heads));
  box[row] = static_cast<cuuint32_t>(box_rows);
  return fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, one, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS
             ? 0
             : -4;
}

template <int ND>
int launch(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, const Dev& p, cudaStream_t st) {
  static bool once = false;
  if (!once) {
    if (cudaFuncSetAttribute(talk_prompt_kernel<ND>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg<ND>::kSmem) != cudaSuccess) return -2;
    once = true;
  }
  int sms = 0, dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) return -2;
  talk_prompt_kernel<ND><<<std::min(p.items, sms), kThreads, Cfg<ND>::kSmem, st>>>(q, k, v, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace

extern "C" int nx_talk_prompt(const NxTalkPromptArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->status == nullptr || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || !(a->scale > 0.0f)) return -1;
  if (a->dim <= 0 || a->dim > 128 || (a->dim & 15) || a->vdim <= 0 || a->vdim > 128 || (a->vdim & 7) || a->chunk < 0) return -1;
  if ((a->ldq | a->ldk | a->ldv | a->ldo) & 7) return -1;
  for (const void* ptr : {a->q, a->k, a->v, static_cast<const void*>(a->out), static_cast<const void*>(a->blocks)})
    if (ptr == nullptr || (reinterpret_cast<uintptr_t>(ptr) & 15)) return -1;
  if (a->bias != nullptr && (a->bias_len <= 0 || a->bias_pitch < NX_TALK_BIAS_NEAR + a->bias_len + NX_TALK_BIAS_FAR || (a->bias_pitch & 3) ||
                             a->bias_pitch > kBiasTable || (reinterpret_cast<uintptr_t>(a->bias) & 15)))
    return -1;
  if (a->n_blocks <= 0) return 0;
  CUtensorMap q, k, v;
  int rc;
  Dev p{};
  p.slabs = a->vdim <= 64 ? 1 : 2;
  p.at_once = std::min(kSlabs / p.slabs, a->kv_heads);
  p.passes = (a->kv_heads + p.at_once - 1) / p.at_once;
  if ((rc = head_map(&q, a->q, a->dim, a->heads, a->q_rows, a->ldq, 128, 0))) return rc;
  if ((rc = head_map(&k, a->k, a->dim, a->kv_heads, a->kv_rows, a->ldk, kKeys, 0))) return rc;
  if ((rc = head_map(&v, a->v, a->vdim, a->kv_heads, a->kv_rows, a->ldv, kKeys, p.at_once))) return rc;
  p.blocks = a->blocks;
  p.bias = a->bias;
  p.out = static_cast<__nv_bfloat16*>(a->out);
  p.status = a->status;
  p.ldo = a->ldo;
  p.heads = a->heads;
  p.kv_heads = a->kv_heads;
  p.rep = a->heads / a->kv_heads;
  p.vdim = a->vdim;
  p.window = a->window;
  p.chunk = a->chunk;
  p.bias_len = a->bias_len;
  p.bias_pitch = a->bias_pitch;
  p.wide_store = (a->ldo % 16 == 0 && a->vdim % 16 == 0 && (reinterpret_cast<uintptr_t>(a->out) & 31) == 0) ? 1 : 0;
  const int64_t items = static_cast<int64_t>(a->n_blocks) * 2 * a->heads * p.passes;
  if (items > 0x3fffffff) return -1;
  p.items = static_cast<int>(items);
  p.scale = a->scale;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->dim <= 64 ? launch<1>(q, k, v, p, st) : launch<2>(q, k, v, p, st);
}
