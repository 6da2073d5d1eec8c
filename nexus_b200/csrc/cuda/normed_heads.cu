// Around the products of attention on normed queries and keys (see nx_api_mixers.h): what lies between the projections and the
// scores, and the mixture of the heads after them.  FP32 arithmetic; activations are read and written in BF16 or FP32.
#include "common.cuh"
#include "mixer_common.cuh"
#include "nx_api_mixers.h"

#include <algorithm>

namespace {
using namespace nx;

// ------------------------------------------------------------------------------------------------
// norms of queries, keys and values, the query's factors, cache append, gate: one block per row
// ------------------------------------------------------------------------------------------------
// `group`: lanes that share a head in the sums
template <typename T, int V>
__global__ void __launch_bounds__(256) head_prep_kernel(const NxHeadPrepArgs a, int group) {
  extern __shared__ __align__(16) float s_inv[];       // [heads + 2 kv_heads]: factor of every head of q, k and v
  const int64_t r = blockIdx.x;
  T* row = static_cast<T*>(a.proj) + r * a.ld;
  const int H = a.heads, G = a.kv_heads, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int normed = H + G, all = normed + (a.unit_values ? G : 0);
  const int per_warp = 32 / group, in_group = lane % group;
  for (int u0 = warp * per_warp; u0 < all; u0 += warps * per_warp) {   // sums of squares; padding columns are zeros
    const int u = u0 + lane / group;
    float ss = 0.0f;
    if (u < all) {
      const T* p = row + (u < H ? a.q_off + u * a.dim : u < normed ? a.k_off + (u - H) * a.dim : a.v_off + (u - normed) * a.vdim);
      const int size = u < normed ? a.dim : a.vdim;
      for (int c = in_group * V; c < size; c += group * V) {
        float v[V];
        load_vec<T, V>(p + c, v);
#pragma unroll
        for (int j = 0; j < V; ++j) ss += v[j] * v[j];
      }
    }
    for (int o = group / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (in_group == 0 && u < all) s_inv[u] = ss;
  }
  __syncthreads();
  float temp = 1.0f;
  if (a.every > 0) temp = 1.0f + a.coef * logf(static_cast<float>((a.positions[r] + 1) / a.every + 1));
  float whole_q = 0.0f, whole_k = 0.0f;
  if (a.norm_all) {                                      // every thread adds up the heads in the same order
    for (int h = 0; h < H; ++h) whole_q += s_inv[h];
    for (int h = 0; h < G; ++h) whole_k += s_inv[H + h];
    __syncthreads();
  }
  for (int u = threadIdx.x; u < all; u += blockDim.x) {
    float ss = s_inv[u], n = static_cast<float>(u < normed ? a.norm_dim : a.norm_vdim);
    if (a.norm_all && u < normed) {
      ss = u < H ? whole_q : whole_k;
      n *= static_cast<float>(u < H ? H : G);
    }
    float f = 1.0f / sqrtf(ss / n + a.eps);
    if (u < H) f *= temp * a.q_scale * (a.head_scale != nullptr ? a.head_scale[u] : 1.0f);
    s_inv[u] = f;
  }
  __syncthreads();
  const int nq = H * a.dim, nk = G * a.dim, nv = G * a.vdim;
  const int64_t slot = a.slots[r];
  T* kc = slot >= 0 ? static_cast<T*>(a.k_cache) + slot * nk : nullptr;
  T* vc = slot >= 0 ? static_cast<T*>(a.v_cache) + slot * nv : nullptr;
  for (int i = threadIdx.x * V; i < nq + nk; i += blockDim.x * V) {
    const bool is_k = i >= nq;
    const int c = is_k ? i - nq : i, h = c / a.dim;
    T* p = row + (is_k ? a.k_off : a.q_off) + c;
    float v[V], w[V];
    load_vec<T, V>(p, v);
    load_vec<float, V>((is_k ? a.w_k : a.w_q) + (a.norm_all ? c : c - h * a.dim), w);
    const float f = s_inv[is_k ? H + h : h];
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] *= f * w[j];
    if (!is_k || a.store_kv) store_vec<T, V>(p, v);
    if (is_k && kc != nullptr) store_vec<T, V>(kc + c, v);
  }
  for (int c = threadIdx.x * V; c < nv; c += blockDim.x * V) {
    T* p = row + a.v_off + c;
    float v[V];
    load_vec<T, V>(p, v);
    if (a.unit_values) {
      const float f = s_inv[normed + c / a.vdim];
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] *= f;
      if (a.store_kv) store_vec<T, V>(p, v);
    }
    if (vc != nullptr) store_vec<T, V>(vc + c, v);
  }
  if (a.gate == nullptr) return;
  for (int h = threadIdx.x; h < H; h += blockDim.x) a.gate[r * H + h] = sigmoid_exact(Num<T>::load(row + a.g_off + h));
}

// ------------------------------------------------------------------------------------------------
// out_h = gate_h sum_g talk[h][g] wide[g][KV head of h]: a thread owns V adjacent columns of one KV head's values and forms all
// query heads of that KV head, N at a time; a group of N mixture factors is one or two vector loads
// ------------------------------------------------------------------------------------------------
constexpr int kMixAhead = 8;       // rows of `wide` in flight per thread

template <typename T, int V, int N>
__global__ void __launch_bounds__(256)
head_mix_kernel(const T* __restrict__ wide, int64_t ldw, const float* __restrict__ talk, const float* __restrict__ gate,
                T* __restrict__ out, int64_t ldo, int rows, int heads, int kv_heads, int vdim) {
  extern __shared__ __align__(16) float s_talk[];       // [KV head][group of N heads][from head][N]
  const int rep = heads / kv_heads, groups = (rep + N - 1) / N, cols = kv_heads * vdim;
  for (int i = threadIdx.x + threadIdx.y * blockDim.x; i < kv_heads * groups * heads * N; i += blockDim.x * blockDim.y) {
    const int k = i % N, g = i / N % heads, grp = i / (N * heads) % groups, c = i / (N * heads * groups), h = grp * N + k;
    s_talk[i] = h < rep ? talk[(c * rep + h) * heads + g] : 0.0f;
  }
  __syncthreads();
  for (int64_t r = blockIdx.x * static_cast<int64_t>(blockDim.y) + threadIdx.y; r < rows;
       r += static_cast<int64_t>(gridDim.x) * blockDim.y) {
    for (int i = threadIdx.x * V; i < cols; i += blockDim.x * V) {
      const int c = i / vdim, d = i % vdim;
      const T* src = wide + r * ldw + i;
      for (int grp = 0; grp < groups; ++grp) {
        const float* t = s_talk + static_cast<int64_t>(c * groups + grp) * heads * N;
        float acc[N][V];
#pragma unroll
        for (int k = 0; k < N; ++k)
#pragma unroll
          for (int j = 0; j < V; ++j) acc[k][j] = 0.0f;
        for (int g0 = 0; g0 < heads; g0 += kMixAhead) {
          uint4 raw[kMixAhead];                           // V elements of T each
#pragma unroll
          for (int u = 0; u < kMixAhead; ++u) {
            const T* p = src + static_cast<int64_t>(min(g0 + u, heads - 1)) * cols;
            if constexpr (V * sizeof(T) == 16) raw[u] = __ldcs(reinterpret_cast<const uint4*>(p));
            else *reinterpret_cast<T*>(&raw[u]) = *p;
          }
#pragma unroll
          for (int u = 0; u < kMixAhead; ++u) {
            if (g0 + u >= heads) break;
            const T* e = reinterpret_cast<const T*>(&raw[u]);
            float f[N];
#pragma unroll
            for (int k = 0; k < N; k += 4) *reinterpret_cast<float4*>(f + k) = *reinterpret_cast<const float4*>(t + (g0 + u) * N + k);
#pragma unroll
            for (int j = 0; j < V; ++j) {
              const float v = Num<T>::load(e + j);
#pragma unroll
              for (int k = 0; k < N; ++k) acc[k][j] = fmaf(f[k], v, acc[k][j]);
            }
          }
        }
#pragma unroll
        for (int k = 0; k < N; ++k) {
          const int h = c * rep + grp * N + k;
          if (grp * N + k >= rep) break;
          const float w = gate != nullptr ? gate[r * heads + h] : 1.0f;
#pragma unroll
          for (int j = 0; j < V; ++j) acc[k][j] *= w;
          store_vec<T, V>(out + r * ldo + static_cast<int64_t>(h) * vdim + d, acc[k]);
        }
      }
    }
  }
}

}  // namespace

extern "C" int nx_head_prep(const NxHeadPrepArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0) return -1;
  if (a->norm_dim <= 0 || a->norm_dim > a->dim || a->norm_vdim <= 0 || a->norm_vdim > a->vdim || a->heads > 1024) return -1;
  if (a->w_q == nullptr || a->w_k == nullptr || a->slots == nullptr || a->k_cache == nullptr || a->v_cache == nullptr) return -1;
  if (a->every > 0 && a->positions == nullptr) return -1;
  if (a->rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const int v16 = a->dtype == NX_BF16 ? 8 : 4;
  const bool vec = ((a->dim | a->vdim | a->q_off | a->k_off | a->v_off | static_cast<int>(a->ld)) & (v16 - 1)) == 0 && al(a->proj) &&
                   al(a->w_q) && al(a->w_k) && al(a->k_cache) && al(a->v_cache);
  const int chunks = (a->heads * a->dim + a->kv_heads * (a->dim + a->vdim)) / (vec ? v16 : 1);
  const int threads = std::max(64, std::min(256, (chunks / 2 + 31) / 32 * 32));
  const size_t smem = static_cast<size_t>(a->heads + 2 * a->kv_heads) * sizeof(float);
  int group = 32;
  while (group > 1 && group / 2 * (vec ? v16 : 1) >= std::max(a->dim, a->vdim)) group /= 2;
  if (a->dtype == NX_BF16) {
    if (vec) head_prep_kernel<__nv_bfloat16, 8><<<a->rows, threads, smem, st>>>(*a, group);
    else head_prep_kernel<__nv_bfloat16, 1><<<a->rows, threads, smem, st>>>(*a, group);
  } else if (a->dtype == NX_F32) {
    if (vec) head_prep_kernel<float, 4><<<a->rows, threads, smem, st>>>(*a, group);
    else head_prep_kernel<float, 1><<<a->rows, threads, smem, st>>>(*a, group);
  } else {
    return -1;
  }
  return launch_status();
}

extern "C" int nx_head_mix(const void* wide, int64_t ldw, const float* talk, const float* gate, void* out, int64_t ldo, int rows,
                           int heads, int kv_heads, int vdim, int dtype, nx_stream_t stream) {
  if (wide == nullptr || talk == nullptr || out == nullptr || heads <= 0 || heads > 96 || kv_heads <= 0 || heads % kv_heads || vdim <= 0)
    return -1;
  if (ldw < static_cast<int64_t>(heads) * kv_heads * vdim || ldo < static_cast<int64_t>(heads) * vdim) return -1;
  if (rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int v16 = dtype == NX_BF16 ? 8 : 4, n = heads / kv_heads <= 4 ? 4 : 8, groups = (heads / kv_heads + n - 1) / n;
  const bool vec = vdim % v16 == 0 && ldw % v16 == 0 && ldo % v16 == 0 &&
                   ((reinterpret_cast<uintptr_t>(wide) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  const int work = kv_heads * vdim / (vec ? v16 : 1);
  const int tx = std::max(32, std::min(256, (work + 31) / 32 * 32)), ty = std::max(1, 256 / tx);
  const dim3 threads(tx, ty);
  const int blocks = std::min((rows + ty - 1) / ty, kNumSmsB200 * 8);
  const int smem = kv_heads * groups * n * heads * static_cast<int>(sizeof(float));
#define NX_HM(T_, V_, N_)                                                                                                       \
  do {                                                                                                                          \
    if (smem > 40 * 1024 &&                                                                                                     \
        cudaFuncSetAttribute(head_mix_kernel<T_, V_, N_>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)    \
      return -2;                                                                                                                \
    head_mix_kernel<T_, V_, N_><<<blocks, threads, smem, st>>>((const T_*)wide, ldw, talk, gate, (T_*)out, ldo, rows, heads,    \
                                                               kv_heads, vdim);                                                 \
  } while (0)
  if (dtype == NX_BF16) {
    if (vec) { if (n == 4) NX_HM(__nv_bfloat16, 8, 4); else NX_HM(__nv_bfloat16, 8, 8); }
    else if (n == 4) NX_HM(__nv_bfloat16, 1, 4);
    else NX_HM(__nv_bfloat16, 1, 8);
  } else if (dtype == NX_F32) {
    if (vec) { if (n == 4) NX_HM(float, 4, 4); else NX_HM(float, 4, 8); }
    else if (n == 4) NX_HM(float, 1, 4);
    else NX_HM(float, 1, 8);
  } else {
    return -1;
  }
#undef NX_HM
  return launch_status();
}
