// Memory-bound building blocks of decoders with heterogeneous layers (see nx_api_mixers.h): the chain "add the normed
// sublayer output, norm for the next sublayer", rotary embedding fused with the paged cache append, the short causal
// convolution with its carried tail (alone, or with rotation and append), low-rank decays, gated norms, the per-layer token
// input, gated activations and logit soft-capping.
// Everything is computed in FP32; activations are read and written in BF16 or FP32.
#include "common.cuh"
#include "mixer_common.cuh"
#include "nx_api_mixers.h"

#include <algorithm>

namespace {
using namespace nx;

// ------------------------------------------------------------------------------------------------
// residual chain: one block per row, the row stays in shared memory between the passes
// ------------------------------------------------------------------------------------------------
template <typename T, int V>
__global__ void residual_norm_kernel(const NxResidualNormArgs a) {
  extern __shared__ __align__(16) float s_row[];
  __shared__ float s_red[32];
  const int64_t r = blockIdx.x;
  const int cols = a.cols;
  float* xr = a.x + r * cols;
  const float inv_cols = 1.0f / static_cast<float>(cols);
  float ss = 0.0f;
  if (a.table != nullptr) {
    const T* e = static_cast<const T*>(a.table) + static_cast<int64_t>(a.tokens[r]) * cols;
    for (int c = threadIdx.x * V; c < cols; c += blockDim.x * V) {
      float v[V];
      load_vec<T, V>(e + c, v);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] *= a.embed_scale;
      if (a.pos_table != nullptr) {
        float p[V];
        load_vec<T, V>(static_cast<const T*>(a.pos_table) + static_cast<int64_t>(a.positions[r]) * cols + c, p);
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] += p[j];
      }
      store_vec<float, V>(xr + c, v);
      store_vec<float, V>(s_row + c, v);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += v[j] * v[j];
    }
  } else if (a.y != nullptr || a.experts != nullptr) {
    const T* yr = static_cast<const T*>(a.y) + r * a.ldy;
    const float yg = a.y_gate != nullptr ? a.y_gate[r] : 1.0f;
    float sy = 0.0f;
    for (int c = threadIdx.x * V; c < cols; c += blockDim.x * V) {
      float v[V];
      if (a.experts != nullptr) {
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] = 0.0f;
        for (int k = 0; k < a.top; ++k) {
          float u[V];
          load_vec<T, V>(static_cast<const T*>(a.experts) + static_cast<int64_t>(a.expert_slots[r * a.top + k]) * a.ld_experts + c, u);
          const float w = a.expert_weights != nullptr ? a.expert_weights[r * a.top + k] : 1.0f;
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] += w * u[j];
        }
        if (a.y != nullptr) {
          float u[V];
          load_vec<T, V>(yr + c, u);
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] = v[j] * a.expert_scale + u[j] * yg;
        } else {
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] *= a.expert_scale;
        }
      } else {
        load_vec<T, V>(yr + c, v);
      }
      if (a.w_post == nullptr) {            // the output is added as it is
        float xv[V];
        load_vec<float, V>(xr + c, xv);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          v[j] = xv[j] + a.res_mult * v[j];
          ss += v[j] * v[j];
        }
        store_vec<float, V>(xr + c, v);
        store_vec<float, V>(s_row + c, v);
        continue;
      }
      store_vec<float, V>(s_row + c, v);
#pragma unroll
      for (int j = 0; j < V; ++j) sy += v[j] * v[j];
    }
    const float inv = a.w_post != nullptr ? a.res_mult / sqrtf(block_sum(sy, s_red) * inv_cols + a.eps) : 0.0f;
    for (int c = threadIdx.x * V; c < cols && a.w_post != nullptr; c += blockDim.x * V) {   // each thread re-reads its own columns
      float v[V], xv[V], w[V];
      load_vec<float, V>(s_row + c, v);
      load_vec<float, V>(xr + c, xv);
      load_vec<float, V>(a.w_post + c, w);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        v[j] = xv[j] + v[j] * inv * w[j];
        ss += v[j] * v[j];
      }
      store_vec<float, V>(xr + c, v);
      store_vec<float, V>(s_row + c, v);
    }
  } else {
    for (int c = threadIdx.x * V; c < cols; c += blockDim.x * V) {
      float v[V];
      load_vec<float, V>(xr + c, v);
      store_vec<float, V>(s_row + c, v);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += v[j] * v[j];
    }
  }
  if (a.x_cast != nullptr) {
    T* o = static_cast<T*>(a.x_cast) + r * a.ldh;
    for (int c = threadIdx.x * V; c < cols; c += blockDim.x * V) {
      float v[V];
      load_vec<float, V>(s_row + c, v);
      store_vec<T, V>(o + c, v);
    }
    for (int c = cols + threadIdx.x; c < a.ldh; c += blockDim.x) Num<T>::store(o + c, 0.0f);
  }
  if (a.scatter != nullptr) {
    for (int k = 0; k < a.top; ++k) {
      T* o = static_cast<T*>(a.scatter) + static_cast<int64_t>(a.scatter_slots[r * a.top + k]) * a.ldh;
      for (int c = threadIdx.x * V; c < cols; c += blockDim.x * V) {
        float v[V];
        load_vec<float, V>(s_row + c, v);
        store_vec<T, V>(o + c, v);
      }
      for (int c = cols + threadIdx.x; c < a.ldh; c += blockDim.x) Num<T>::store(o + c, 0.0f);
    }
  }
  if (a.w_dot != nullptr) {
    float sd = 0.0f;
    for (int c = threadIdx.x * V; c < cols; c += blockDim.x * V) {
      float v[V], w[V];
      load_vec<float, V>(s_row + c, v);
      load_vec<float, V>(a.w_dot + c, w);
#pragma unroll
      for (int j = 0; j < V; ++j) sd += v[j] * w[j];
    }
    sd = block_sum(sd, s_red);
    if (threadIdx.x == 0) a.dot_out[r] = sigmoid_exact(sd);
  }
  if (a.h != nullptr) {
    const float inv = 1.0f / sqrtf(block_sum(ss, s_red) * inv_cols + a.eps);
    T* o = static_cast<T*>(a.h) + r * a.ldh;
    for (int c = threadIdx.x * V; c < cols; c += blockDim.x * V) {
      float v[V], w[V];
      load_vec<float, V>(s_row + c, v);
      load_vec<float, V>(a.w_next + c, w);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] *= inv * w[j];
      store_vec<T, V>(o + c, v);
    }
    for (int c = cols + threadIdx.x; c < a.ldh; c += blockDim.x) Num<T>::store(o + c, 0.0f);
  }
}

// ------------------------------------------------------------------------------------------------
// rotary embedding (rotate-half layout, first rot_dims of a head) + cache append: one block per row
// ------------------------------------------------------------------------------------------------
template <typename T>
__global__ void rope_append_kernel(const NxRopeAppendArgs a) {
  const int64_t r = blockIdx.x;
  const int half = a.rot_dims / 2;
  T* row = static_cast<T*>(a.proj) + r * a.ld;
  const int64_t pos = a.positions[r], slot = a.slots[r];
  const float* cs = a.cos_t + pos * half;
  const float* sn = a.sin_t + pos * half;
  T* kc = static_cast<T*>(a.k_cache) + slot * a.kv_heads * a.dim;
  T* vc = static_cast<T*>(a.v_cache) + slot * a.kv_heads * a.vdim;
  const int nq = a.heads * half, nk = a.kv_heads * half;
  for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
    const bool is_k = i >= nq;
    const int u = is_k ? i - nq : i;
    const int h = u / half, j = u % half;
    T* p = row + (is_k ? a.k_off : a.q_off) + h * a.dim + j;
    const float x0 = Num<T>::load(p), x1 = Num<T>::load(p + half), c = cs[j], s = sn[j];
    const float y0 = x0 * c - x1 * s, y1 = x1 * c + x0 * s;
    Num<T>::store(p, y0);
    Num<T>::store(p + half, y1);
    if (is_k && slot >= 0) {
      Num<T>::store(kc + h * a.dim + j, y0);
      Num<T>::store(kc + h * a.dim + j + half, y1);
    }
  }
  if (slot < 0) return;
  const int rest = a.dim - a.rot_dims;
  for (int i = threadIdx.x; i < a.kv_heads * rest; i += blockDim.x) {
    const int o = (i / rest) * a.dim + a.rot_dims + i % rest;
    kc[o] = row[a.k_off + o];
  }
  for (int i = threadIdx.x; i < a.kv_heads * a.vdim; i += blockDim.x) vc[i] = row[a.v_off + i];
}

// ------------------------------------------------------------------------------------------------
// latent attention: norms of both latents, rotation of the shared key part, cache append, gate; one block per row
// ------------------------------------------------------------------------------------------------
template <typename T, int V>
__device__ __forceinline__ float sum_squares(const T* p, int n) {
  float ss = 0.0f;
  for (int c = threadIdx.x * V; c < n; c += blockDim.x * V) {
    float v[V];
    load_vec<T, V>(p + c, v);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += v[j] * v[j];
  }
  return ss;
}

template <typename T, int V>
__global__ void latent_prep_kernel(const NxLatentPrepArgs a) {
  __shared__ float s_red[32];
  const int64_t r = blockIdx.x;
  const T* row = static_cast<const T*>(a.proj) + r * a.ld;
  const int64_t pos = a.positions[r], slot = a.slots[r];
  const T *q = row + a.q_off, *k = row + a.c_off;
  const float inv_q =
      a.q_rank > 0 ? 1.0f / sqrtf(block_sum(sum_squares<T, V>(q, a.q_rank), s_red) / static_cast<float>(a.q_rank) + a.eps) : 0.0f;
  const float inv_k = 1.0f / sqrtf(block_sum(sum_squares<T, V>(k, a.kv_rank), s_red) / static_cast<float>(a.kv_rank) + a.eps);
  T* cq = static_cast<T*>(a.cq) + r * a.ldq;
  for (int c = threadIdx.x * V; c < a.q_rank; c += blockDim.x * V) {
    float v[V], w[V];
    load_vec<T, V>(q + c, v);
    load_vec<float, V>(a.w_q + c, w);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] *= inv_q * w[j];
    store_vec<T, V>(cq + c, v);
  }
  for (int c = a.q_rank + threadIdx.x; c < a.ldq; c += blockDim.x) Num<T>::store(cq + c, 0.0f);
  T* cache = slot >= 0 ? static_cast<T*>(a.cache) + slot * a.ld_cache : nullptr;
  T* lat = a.lat != nullptr ? static_cast<T*>(a.lat) + r * a.ld_cache : nullptr;
  for (int c = threadIdx.x * V; c < a.kv_rank; c += blockDim.x * V) {
    float v[V], w[V];
    load_vec<T, V>(k + c, v);
    load_vec<float, V>(a.w_kv + c, w);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] *= inv_k * w[j];
    if (cache != nullptr) store_vec<T, V>(cache + c, v);
    if (lat != nullptr) store_vec<T, V>(lat + c, v);
  }
  const int half = a.rot_dims / 2;
  for (int j = threadIdx.x; j < half; j += blockDim.x) {
    const float u = Num<T>::load(row + a.r_off + j), v = Num<T>::load(row + a.r_off + half + j);
    const float c = a.cos_t[pos * half + j], s = a.sin_t[pos * half + j];
    const float y0 = u * c - v * s, y1 = v * c + u * s;
    if (cache != nullptr) {
      Num<T>::store(cache + a.rot_col + j, y0);
      Num<T>::store(cache + a.rot_col + half + j, y1);
    }
    if (lat != nullptr) {
      Num<T>::store(lat + a.rot_col + j, y0);
      Num<T>::store(lat + a.rot_col + half + j, y1);
    }
  }
  if (lat != nullptr) {
    for (int c = a.kv_rank + threadIdx.x; c < a.rot_col; c += blockDim.x) Num<T>::store(lat + c, 0.0f);
    for (int c = a.rot_col + a.rot_dims + threadIdx.x; c < a.ld_cache; c += blockDim.x) Num<T>::store(lat + c, 0.0f);
  }
  if (a.gate == nullptr) return;
  for (int h = threadIdx.x; h < a.heads; h += blockDim.x)
    a.gate[r * a.heads + h] = sigmoid_exact(Num<T>::load(row + a.g_off + h));
}

// V adjacent pairs per thread; a block takes blockDim.y rows
template <typename T, int V>
__global__ void rope_heads_kernel(const T* __restrict__ src, int64_t ld_src, int src_head, int src_off, T* dst, int64_t ld_dst,
                                  int dst_head, int dst_off, int rows, int heads, int rot_dims, int width,
                                  const int32_t* __restrict__ positions, const float* __restrict__ cos_t,
                                  const float* __restrict__ sin_t) {
  const int64_t r = blockIdx.x * static_cast<int64_t>(blockDim.y) + threadIdx.y;
  if (r >= rows) return;
  const int half = rot_dims / 2, per = half / V;
  const int64_t pos = positions[r];
  for (int i = threadIdx.x; i < heads * per; i += blockDim.x) {
    const int h = i / per, j = (i % per) * V;
    const T* s = src + r * ld_src + static_cast<int64_t>(h) * src_head + src_off + j;
    T* d = dst + r * ld_dst + static_cast<int64_t>(h) * dst_head + dst_off + j;
    float u[V], v[V], c[V], sn[V];
    load_vec<T, V>(s, u);
    load_vec<T, V>(s + half, v);
    load_vec<float, V>(cos_t + pos * half + j, c);
    load_vec<float, V>(sin_t + pos * half + j, sn);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const float a = u[k] * c[k] - v[k] * sn[k];
      v[k] = v[k] * c[k] + u[k] * sn[k];
      u[k] = a;
    }
    store_vec<T, V>(d, u);
    store_vec<T, V>(d + half, v);
  }
  const int rest = width - rot_dims;
  for (int i = threadIdx.x; i < heads * rest; i += blockDim.x)
    Num<T>::store(dst + r * ld_dst + static_cast<int64_t>(i / rest) * dst_head + dst_off + rot_dims + i % rest, 0.0f);
}

// ------------------------------------------------------------------------------------------------
// causal convolution + SiLU.  A thread owns V adjacent channels over one tile of a segment's tokens;
// the first tile reads the carried tail and is the one that writes the new one, so that no other
// block touches the tail of this segment.
// ------------------------------------------------------------------------------------------------
constexpr int kConvTile = 32;

// emit(row, token of the segment, sums of V channels) for every token of the tile
template <typename T, int TAPS, int V, typename Emit>
__device__ __forceinline__ void conv_tile(const NxConvArgs& a, Emit emit) {
  const int sg = blockIdx.z;
  const int len = a.seg.len[sg];
  const int t0 = blockIdx.y * kConvTile;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (t0 >= len || c >= a.channels) return;
  const int64_t row0 = a.seg.row0[sg];
  constexpr int HIST = TAPS > 1 ? TAPS - 1 : 1;
  float w[TAPS][V], hist[HIST][V], bias[V];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) load_vec<float, V>(a.w + static_cast<int64_t>(j) * a.channels + c, w[j]);
#pragma unroll
  for (int v = 0; v < V; ++v) bias[v] = a.bias != nullptr ? a.bias[c + v] : 0.0f;
  const T* x = static_cast<const T*>(a.x) + row0 * a.ldx + c;
  T* st = static_cast<T*>(a.state) + static_cast<int64_t>(a.seg.seq[sg]) * (TAPS - 1) * a.channels + c;
  const bool carried = a.seg.pos[sg] > 0;
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int t = t0 - (TAPS - 1) + j;     // token of the segment this tap's first input is
    if (t >= 0) {
      load_vec<T, V>(x + static_cast<int64_t>(t) * a.ldx, hist[j]);
    } else if (carried) {                  // only in the first tile: kConvTile >= TAPS - 1
      load_vec<T, V>(st + static_cast<int64_t>(TAPS - 1 + t) * a.channels, hist[j]);
    } else {
#pragma unroll
      for (int v = 0; v < V; ++v) hist[j][v] = 0.0f;
    }
  }
  if (t0 == 0) {
    float tail[HIST][V];
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      const int t = len - (TAPS - 1) + j;
      if (t >= 0) {
        load_vec<T, V>(x + static_cast<int64_t>(t) * a.ldx, tail[j]);
      } else if (carried) {                // a segment shorter than the tail keeps the newest of the old inputs
        load_vec<T, V>(st + static_cast<int64_t>(TAPS - 1 + t) * a.channels, tail[j]);
      } else {
#pragma unroll
        for (int v = 0; v < V; ++v) tail[j][v] = 0.0f;
      }
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) store_vec<T, V>(st + static_cast<int64_t>(j) * a.channels, tail[j]);
  }
  const int t1 = min(len, t0 + kConvTile);
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    float cur[V], acc[V];
    load_vec<T, V>(x + static_cast<int64_t>(t) * a.ldx, cur);
#pragma unroll
    for (int v = 0; v < V; ++v) acc[v] = bias[v] + w[TAPS - 1][v] * cur[v];
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
      for (int v = 0; v < V; ++v) acc[v] += w[j][v] * hist[j][v];
    emit(row0 + t, t, acc);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
      for (int v = 0; v < V; ++v) hist[j][v] = j + 1 < TAPS - 1 ? hist[j + 1 < HIST ? j + 1 : j][v] : cur[v];
  }
}

template <typename T, int TAPS, int V>
__global__ void conv_silu_kernel(const NxConvArgs a) {
  T* y = static_cast<T*>(a.y) + (blockIdx.x * blockDim.x + threadIdx.x) * V;
  conv_tile<T, TAPS, V>(a, [&](int64_t row, int, float (&acc)[V]) {
#pragma unroll
    for (int v = 0; v < V; ++v) acc[v] = sizeof(T) == 4 ? silu_exact(acc[v]) : acc[v] * __fdividef(1.0f, 1.0f + __expf(-acc[v]));
    store_vec<T, V>(y + row * a.ldy, acc);
  });
}

// convolution + rotation of neighbouring pairs + value mixing + cache append: a thread's V channels lie in one head
template <typename T, int TAPS, int V>
__global__ void conv_rope_kernel(const NxConvRopeArgs a) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim, half = a.rot_dims / 2;
  const int part = c < nq ? 0 : c < nq + nk ? 1 : 2;                  // q, k, v
  const int u = part == 0 ? c : part == 1 ? c - nq : c - nq - nk;     // column inside the part
  const int d = part < 2 ? u % a.dim : 0;
  T* y = static_cast<T*>(a.conv.y) + c;
  T* first = static_cast<T*>(a.first) + u;
  const float mix = a.mix != nullptr ? *a.mix : 0.0f;
  const int pos0 = a.conv.seg.pos[blockIdx.z];
  conv_tile<T, TAPS, V>(a.conv, [&](int64_t row, int t, float (&acc)[V]) {
    const int64_t slot = part > 0 ? a.slots[row] : -1;
    if (part < 2) {
      const int64_t at = static_cast<int64_t>(pos0 + t) * half + d / 2;
#pragma unroll
      for (int v = 0; v < V; v += 2)
        if (d + v < a.rot_dims) {
          const float cs = a.cos_t[at + v / 2], sn = a.sin_t[at + v / 2], p = acc[v], q = acc[v + 1];
          acc[v] = p * cs - q * sn;
          acc[v + 1] = q * cs + p * sn;
        }
      if (part == 1 && slot >= 0) store_vec<T, V>(static_cast<T*>(a.k_cache) + slot * nk + u, acc);
    } else {
      if (a.mix != nullptr) {
        float f[V];
        load_vec<T, V>(first + row * nv, f);
#pragma unroll
        for (int v = 0; v < V; ++v) acc[v] = (1.0f - mix) * acc[v] + mix * f[v];
      } else if (a.first != nullptr) {
        store_vec<T, V>(first + row * nv, acc);
      }
      if (slot >= 0) store_vec<T, V>(static_cast<T*>(a.v_cache) + slot * nv + u, acc);
    }
    if (part == 0 || a.store_kv) store_vec<T, V>(y + row * a.conv.ldy, acc);
  });
}

// ------------------------------------------------------------------------------------------------
// gated norm: a warp (small groups) or a block (large groups) per (row, group)
// ------------------------------------------------------------------------------------------------
constexpr int kGatedWarpCols = 512;

template <typename T, bool kWarp>
__global__ void gated_norm_kernel(const NxGatedNormArgs a) {
  __shared__ float s_red[32];
  const int lanes = kWarp ? 32 : blockDim.x;
  const int64_t item = kWarp ? blockIdx.x * static_cast<int64_t>(blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.x;
  if (item >= static_cast<int64_t>(a.rows) * a.groups) return;   // whole warps (or blocks) leave together
  const int lane = kWarp ? threadIdx.x & 31 : threadIdx.x;
  const int64_t r = item / a.groups;
  const int g = static_cast<int>(item % a.groups), n = a.group_size;
  const T* y = static_cast<const T*>(a.y) + r * a.ldy + static_cast<int64_t>(g) * n;
  const T* z = static_cast<const T*>(a.z) + r * a.ldz + static_cast<int64_t>(g) * n;
  T* o = static_cast<T*>(a.out) + r * a.ldo + static_cast<int64_t>(g) * n;
  const float* w = a.w + (a.w_shared ? 0 : static_cast<int64_t>(g) * n);
  float ss = 0.0f;
  for (int c = lane; c < n; c += lanes) {
    float v = Num<T>::load(y + c);
    if (a.gate_first) v *= silu_exact(Num<T>::load(z + c));
    ss += v * v;
  }
  ss = kWarp ? warp_sum(ss) : block_sum(ss, s_red);
  const float inv = a.out_scale / sqrtf(ss / static_cast<float>(n) + a.eps);
  for (int c = lane; c < n; c += lanes)
    Num<T>::store(o + c, Num<T>::load(y + c) * silu_exact(Num<T>::load(z + c)) * inv * w[c]);
}

// the same with vector accesses and the gated values kept in registers: groups of up to 16 values per thread
template <typename T, int V, bool kWarp>
__global__ void gated_norm_vec_kernel(const NxGatedNormArgs a) {
  constexpr int kIter = 16 / V;
  __shared__ float s_red[32];
  const int lanes = kWarp ? 32 : blockDim.x;
  const int64_t item = kWarp ? blockIdx.x * static_cast<int64_t>(blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.x;
  if (item >= static_cast<int64_t>(a.rows) * a.groups) return;
  const int lane = kWarp ? threadIdx.x & 31 : threadIdx.x;
  const int64_t r = item / a.groups;
  const int g = static_cast<int>(item % a.groups), n = a.group_size;
  const T* y = static_cast<const T*>(a.y) + r * a.ldy + static_cast<int64_t>(g) * n;
  const T* z = static_cast<const T*>(a.z) + r * a.ldz + static_cast<int64_t>(g) * n;
  T* o = static_cast<T*>(a.out) + r * a.ldo + static_cast<int64_t>(g) * n;
  const float* w = a.w + (a.w_shared ? 0 : static_cast<int64_t>(g) * n);
  float v[kIter][V], ss = 0.0f;
#pragma unroll
  for (int i = 0; i < kIter; ++i) {
    const int c = (lane + i * lanes) * V;
    if (c < n) {
      float zv[V];
      load_vec<T, V>(y + c, v[i]);
      load_vec<T, V>(z + c, zv);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const float gate = zv[j] * __fdividef(1.0f, 1.0f + __expf(-zv[j])), u = v[i][j] * gate;
        ss += a.gate_first ? u * u : v[i][j] * v[i][j];
        v[i][j] = u;
      }
    }
  }
  ss = kWarp ? warp_sum(ss) : block_sum(ss, s_red);
  const float inv = a.out_scale / sqrtf(ss / static_cast<float>(n) + a.eps);
#pragma unroll
  for (int i = 0; i < kIter; ++i) {
    const int c = (lane + i * lanes) * V;
    if (c < n) {
      float wv[V];
      load_vec<float, V>(w + c, wv);
#pragma unroll
      for (int j = 0; j < V; ++j) v[i][j] *= inv * wv[j];
      store_vec<T, V>(o + c, v[i]);
    }
  }
}

// ------------------------------------------------------------------------------------------------
// elementwise
// ------------------------------------------------------------------------------------------------
template <typename T>
__global__ void token_side_kernel(const float* __restrict__ a, int64_t lda, const int32_t* __restrict__ tokens,
                                  const T* __restrict__ table, int64_t ld_table, int offset, T* __restrict__ out,
                                  int64_t ldo, int dim, int rows) {
  const int64_t r = blockIdx.x * static_cast<int64_t>(blockDim.y) + threadIdx.y;
  if (r >= rows) return;
  const T* e = table + static_cast<int64_t>(tokens[r]) * ld_table + offset;
  for (int j = threadIdx.x; j < ldo; j += blockDim.x) {
    float v = 0.0f;
    if (j < dim) v = gelu_tanh_exact(a[r * lda + j]) * Num<T>::load(e + j);
    Num<T>::store(out + r * ldo + j, v);
  }
}

// V == 8 or 1; a column's gate and value: halves of a row, or turns of eight columns (interleaved)
template <typename T, int V>
__global__ void glu_kernel(const T* __restrict__ h, int64_t ldh, T* __restrict__ out, int64_t ldo, int half, int interleaved,
                           const NxGlu f) {
  const int64_t r = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= half) return;
  const T* p = h + r * ldh + (interleaved ? c / 8 * 16 + c % 8 : c);
  float g[V], u[V];
  load_vec<T, V>(p, g);
  load_vec<T, V>(p + (interleaved ? 8 : half), u);
#pragma unroll
  for (int j = 0; j < V; ++j) g[j] = glu_apply<sizeof(T) == 4>(f, g[j], u[j]);
  store_vec<T, V>(out + r * ldo + c, g);
}

__global__ void softcap_kernel(float* __restrict__ x, int64_t ld, int cols, float cap, float scale) {
  float* xr = x + blockIdx.y * ld;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c < cols) xr[c] = cap > 0.0f ? cap * tanhf(scale * xr[c] / cap) : scale * xr[c];
}

// log2 of a decay sigmoid(z)^(1 / tau) with z of low rank: 128 columns x 32 rows per block, 16 rows per thread
constexpr int kDecayCols = 128, kDecayRows = 32, kDecayRank = 16;
template <typename T>
__global__ void __launch_bounds__(256)
decay_gate_kernel(const T* __restrict__ a, int64_t lda, const float* __restrict__ w, const float* __restrict__ bias,
                  float* __restrict__ out, int64_t ldo, int rows, int cols, int rank, float mul) {
  __shared__ float s_w[kDecayRank][kDecayCols + 1];
  __shared__ __align__(16) float s_a[kDecayRows][kDecayRank];
  const int c0 = blockIdx.x * kDecayCols, tx = threadIdx.x % kDecayCols, ty = threadIdx.x / kDecayCols, c = c0 + tx;
  const int64_t r0 = static_cast<int64_t>(blockIdx.y) * kDecayRows;
  float acc[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) acc[i] = 0.0f;
  for (int k0 = 0; k0 < rank; k0 += kDecayRank) {
    __syncthreads();
    for (int i = threadIdx.x; i < kDecayCols * kDecayRank; i += 256) {
      const int col = i / kDecayRank, k = i % kDecayRank;
      s_w[k][col] = c0 + col < cols && k0 + k < rank ? w[static_cast<int64_t>(c0 + col) * rank + k0 + k] : 0.0f;
    }
    for (int i = threadIdx.x; i < kDecayRows * kDecayRank; i += 256) {
      const int row = i / kDecayRank, k = i % kDecayRank;
      s_a[row][k] = r0 + row < rows && k0 + k < rank ? Num<T>::load(a + (r0 + row) * lda + k0 + k) : 0.0f;
    }
    __syncthreads();
    float wk[kDecayRank];
#pragma unroll
    for (int k = 0; k < kDecayRank; ++k) wk[k] = s_w[k][tx];
#pragma unroll
    for (int i = 0; i < 16; ++i)
#pragma unroll
      for (int k = 0; k < kDecayRank; k += 4) {
        const float4 v = *reinterpret_cast<const float4*>(&s_a[ty * 16 + i][k]);     // the same for the whole warp
        acc[i] = fmaf(v.x, wk[k], fmaf(v.y, wk[k + 1], fmaf(v.z, wk[k + 2], fmaf(v.w, wk[k + 3], acc[i]))));
      }
  }
  if (c >= cols) return;
  const float b = bias[c];
#pragma unroll
  for (int i = 0; i < 16; ++i)
    if (r0 + ty * 16 + i < rows) out[(r0 + ty * 16 + i) * ldo + c] = -softplus_exact(-(acc[i] + b)) * mul;
}

bool conv_ok(const NxConvArgs& a) {
  return a.channels > 0 && a.taps >= 1 && a.taps <= 8 && a.seg.count <= 65535 && (a.seg.max_len + kConvTile - 1) / kConvTile <= 65535;
}
template <int V>
dim3 conv_grid(const NxConvArgs& a, int threads) {
  return dim3((a.channels / V + threads - 1) / threads, (a.seg.max_len + kConvTile - 1) / kConvTile, a.seg.count);
}
constexpr int kConvThreads = 128;
#define NX_CONV_TAPS(KERNEL_, CONV_)                                                                             \
  switch ((CONV_).taps) {                                                                                        \
    case 1: KERNEL_<T, 1, V><<<conv_grid<V>(CONV_, kConvThreads), kConvThreads, 0, st>>>(*a); break;             \
    case 2: KERNEL_<T, 2, V><<<conv_grid<V>(CONV_, kConvThreads), kConvThreads, 0, st>>>(*a); break;             \
    case 3: KERNEL_<T, 3, V><<<conv_grid<V>(CONV_, kConvThreads), kConvThreads, 0, st>>>(*a); break;             \
    case 4: KERNEL_<T, 4, V><<<conv_grid<V>(CONV_, kConvThreads), kConvThreads, 0, st>>>(*a); break;             \
    case 5: KERNEL_<T, 5, V><<<conv_grid<V>(CONV_, kConvThreads), kConvThreads, 0, st>>>(*a); break;             \
    case 6: KERNEL_<T, 6, V><<<conv_grid<V>(CONV_, kConvThreads), kConvThreads, 0, st>>>(*a); break;             \
    case 7: KERNEL_<T, 7, V><<<conv_grid<V>(CONV_, kConvThreads), kConvThreads, 0, st>>>(*a); break;             \
    case 8: KERNEL_<T, 8, V><<<conv_grid<V>(CONV_, kConvThreads), kConvThreads, 0, st>>>(*a); break;             \
    default: return -1;                                                                                          \
  }                                                                                                              \
  return launch_status()
template <typename T, int V>
int launch_conv(const NxConvArgs* a, cudaStream_t st) {
  NX_CONV_TAPS(conv_silu_kernel, *a);
}
template <typename T, int V>
int launch_conv_rope(const NxConvRopeArgs* a, cudaStream_t st) {
  NX_CONV_TAPS(conv_rope_kernel, a->conv);
}
#undef NX_CONV_TAPS

template <typename T>
int launch_residual(const NxResidualNormArgs* a, cudaStream_t st) {
  const bool vec = a->cols % 4 == 0 && (a->y == nullptr || a->ldy % 4 == 0) && a->ldh % 4 == 0 &&
                   (a->experts == nullptr || a->ld_experts % 4 == 0);
  const int per = vec ? 4 : 1;
  int threads = ((a->cols / per + 1) / 2 + 31) / 32 * 32;
  threads = std::max(64, std::min(512, threads));
  const size_t smem = static_cast<size_t>(a->cols) * sizeof(float);
  if (smem > 200 * 1024) return -1;
  if (smem > 48 * 1024) {
    const cudaError_t e = vec ? cudaFuncSetAttribute(residual_norm_kernel<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)
                              : cudaFuncSetAttribute(residual_norm_kernel<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return -2;
  }
  if (vec) residual_norm_kernel<T, 4><<<a->rows, threads, smem, st>>>(*a);
  else residual_norm_kernel<T, 1><<<a->rows, threads, smem, st>>>(*a);
  return launch_status();
}

}  // namespace

// ================================================================================================
extern "C" int nx_residual_norm(const NxResidualNormArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->cols <= 0 || a->x == nullptr) return -1;
  if (a->rows <= 0) return 0;
  if (a->experts != nullptr && (a->expert_slots == nullptr || a->top < 1)) return -1;
  if (a->scatter != nullptr && (a->scatter_slots == nullptr || a->top < 1 || a->ldh < a->cols)) return -1;
  if (a->w_dot != nullptr && a->dot_out == nullptr) return -1;
  if (a->h != nullptr && a->w_next == nullptr) return -1;
  if ((a->h != nullptr || a->x_cast != nullptr) && a->ldh < a->cols) return -1;
  if (a->table != nullptr && a->tokens == nullptr) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a->dtype == NX_BF16) return launch_residual<__nv_bfloat16>(a, st);
  if (a->dtype == NX_F32) return launch_residual<float>(a, st);
  return -1;
}

extern "C" int nx_rope_append(const NxRopeAppendArgs* a, nx_stream_t stream) {
  if (a == nullptr) return -1;
  if (a->rows <= 0) return 0;
  if (a->rot_dims < 0 || (a->rot_dims & 1) || a->rot_dims > a->dim) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int work = std::max(a->heads * a->rot_dims / 2, a->kv_heads * std::max(a->dim, a->vdim));
  const int threads = std::max(64, std::min(256, (work + 31) / 32 * 32));
  if (a->dtype == NX_BF16) rope_append_kernel<__nv_bfloat16><<<a->rows, threads, 0, st>>>(*a);
  else if (a->dtype == NX_F32) rope_append_kernel<float><<<a->rows, threads, 0, st>>>(*a);
  else return -1;
  return launch_status();
}

extern "C" int nx_latent_prep(const NxLatentPrepArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->q_rank < 0 || a->kv_rank <= 0 || a->heads <= 0 || a->rot_dims < 0 || (a->rot_dims & 1)) return -1;
  if (a->ldq < a->q_rank || a->rot_col < a->kv_rank || a->ld_cache < a->rot_col + a->rot_dims) return -1;
  if (a->rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = ((a->q_rank | a->kv_rank | a->q_off | a->c_off) & 3) == 0 && ((a->ld | a->ldq | a->ld_cache) & 3) == 0 &&
                   (reinterpret_cast<uintptr_t>(a->proj) & 15) == 0;
  const int most = std::max(a->q_rank, a->kv_rank) / (vec ? 4 : 1);
  const int threads = std::max(64, std::min(256, (most + 31) / 32 * 32));
  if (a->dtype == NX_BF16) {
    if (vec) latent_prep_kernel<__nv_bfloat16, 4><<<a->rows, threads, 0, st>>>(*a);
    else latent_prep_kernel<__nv_bfloat16, 1><<<a->rows, threads, 0, st>>>(*a);
  } else if (a->dtype == NX_F32) {
    if (vec) latent_prep_kernel<float, 4><<<a->rows, threads, 0, st>>>(*a);
    else latent_prep_kernel<float, 1><<<a->rows, threads, 0, st>>>(*a);
  } else {
    return -1;
  }
  return launch_status();
}

extern "C" int nx_rope_heads(const void* src, int64_t ld_src, int src_head, int src_off, void* dst, int64_t ld_dst,
                             int dst_head, int dst_off, int rows, int heads, int rot_dims, int width,
                             const int32_t* positions, const float* cos_t, const float* sin_t, int dtype,
                             nx_stream_t stream) {
  if (rot_dims < 0 || (rot_dims & 1) || width < rot_dims || heads <= 0) return -1;
  if (rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int half = rot_dims / 2;
  const bool vec = half % 8 == 0 && ((ld_src | src_head | src_off | ld_dst | dst_head | dst_off) & 7) == 0 &&
                   ((reinterpret_cast<uintptr_t>(src) | reinterpret_cast<uintptr_t>(dst)) & 15) == 0;
  const int work = std::max(heads * half / (vec ? 8 : 1), 32);
  const int tx = std::min(256, (work + 31) / 32 * 32), ty = 256 / tx;
  const dim3 block(tx, ty), grid((rows + ty - 1) / ty);
#define NX_RH(T_, V_)                                                                                                   \
  rope_heads_kernel<T_, V_><<<grid, block, 0, st>>>(static_cast<const T_*>(src), ld_src, src_head, src_off,             \
                                                    static_cast<T_*>(dst), ld_dst, dst_head, dst_off, rows, heads,      \
                                                    rot_dims, width, positions, cos_t, sin_t)
  if (dtype == NX_BF16) { if (vec) NX_RH(__nv_bfloat16, 8); else NX_RH(__nv_bfloat16, 1); }
  else if (dtype == NX_F32) { if (vec) NX_RH(float, 8); else NX_RH(float, 1); }
  else return -1;
#undef NX_RH
  return launch_status();
}

extern "C" int nx_conv_silu(const NxConvArgs* a, nx_stream_t stream) {
  if (a == nullptr || !conv_ok(*a)) return -1;
  if (a->seg.count <= 0 || a->seg.max_len <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool v2 = a->channels % 2 == 0 && a->ldx % 2 == 0 && a->ldy % 2 == 0 && (reinterpret_cast<uintptr_t>(a->x) & 7) == 0;
  const bool v4 = a->channels % 4 == 0 && a->ldx % 4 == 0 && a->ldy % 4 == 0 && (reinterpret_cast<uintptr_t>(a->x) & 7) == 0 &&
                  (reinterpret_cast<uintptr_t>(a->y) & 7) == 0 && a->taps <= 4;
  if (a->dtype == NX_BF16 && v4) return launch_conv<__nv_bfloat16, 4>(a, st);
  if (a->dtype == NX_BF16) return v2 ? launch_conv<__nv_bfloat16, 2>(a, st) : launch_conv<__nv_bfloat16, 1>(a, st);
  if (a->dtype == NX_F32) return v2 ? launch_conv<float, 2>(a, st) : launch_conv<float, 1>(a, st);
  return -1;
}

extern "C" int nx_conv_rope_append(const NxConvRopeArgs* a, nx_stream_t stream) {
  if (a == nullptr || !conv_ok(a->conv) || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads) return -1;
  if (a->dim <= 0 || a->vdim <= 0 || ((a->dim | a->vdim) & 3) || a->rot_dims < 0 || (a->rot_dims & 1) || a->rot_dims > a->dim) return -1;
  if (a->conv.channels != a->heads * a->dim + a->kv_heads * (a->dim + a->vdim) || ((a->conv.ldx | a->conv.ldy) & 3)) return -1;
  if (a->mix != nullptr && a->first == nullptr) return -1;
  for (const void* p : {a->conv.x, static_cast<const void*>(a->conv.y), static_cast<const void*>(a->k_cache),
                        static_cast<const void*>(a->v_cache), static_cast<const void*>(a->first)})
    if (reinterpret_cast<uintptr_t>(p) & 15) return -1;
  if (a->conv.seg.count <= 0 || a->conv.seg.max_len <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a->conv.dtype == NX_BF16)
    return a->conv.taps <= 4 ? launch_conv_rope<__nv_bfloat16, 4>(a, st) : launch_conv_rope<__nv_bfloat16, 2>(a, st);
  if (a->conv.dtype == NX_F32) return launch_conv_rope<float, 2>(a, st);
  return -1;
}

extern "C" int nx_decay_gate(const void* a, int64_t lda, const float* w, const float* bias, float* out, int64_t ldo, int rows,
                             int cols, int rank, float tau, int dtype, nx_stream_t stream) {
  if (cols <= 0 || rank <= 0 || !(tau > 0.0f) || lda < rank || ldo < cols) return -1;
  if (rows <= 0) return 0;
  if ((rows + kDecayRows - 1) / kDecayRows > 65535) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 grid((cols + kDecayCols - 1) / kDecayCols, (rows + kDecayRows - 1) / kDecayRows);
  const float mul = 1.4426950408889634f / tau;
  if (dtype == NX_BF16)
    decay_gate_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(static_cast<const __nv_bfloat16*>(a), lda, w, bias, out, ldo, rows, cols,
                                                           rank, mul);
  else if (dtype == NX_F32)
    decay_gate_kernel<float><<<grid, 256, 0, st>>>(static_cast<const float*>(a), lda, w, bias, out, ldo, rows, cols, rank, mul);
  else
    return -1;
  return launch_status();
}

extern "C" int nx_gated_norm(const NxGatedNormArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->groups <= 0 || a->group_size <= 0) return -1;
  if (a->rows <= 0) return 0;
  if (a->dtype != NX_BF16 && a->dtype != NX_F32) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int64_t items = static_cast<int64_t>(a->rows) * a->groups;
  if (items > 0x7fffffff) return -1;
  const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  if (a->dtype == NX_BF16 && a->group_size % 8 == 0 && a->ldy % 8 == 0 && a->ldz % 8 == 0 && a->ldo % 8 == 0 && al(a->y) && al(a->z) &&
      al(a->out) && al(a->w) && a->group_size <= 16384) {
    if (a->group_size <= 512) {
      gated_norm_vec_kernel<__nv_bfloat16, 8, true><<<static_cast<int>((items + 7) / 8), 256, 0, st>>>(*a);
    } else {
      const int threads = std::max(64, (a->group_size / 16 + 31) / 32 * 32);
      gated_norm_vec_kernel<__nv_bfloat16, 8, false><<<static_cast<int>(items), threads, 0, st>>>(*a);
    }
    return launch_status();
  }
  if (a->group_size <= kGatedWarpCols) {
    const int blocks = static_cast<int>((items + 7) / 8);
    if (a->dtype == NX_BF16) gated_norm_kernel<__nv_bfloat16, true><<<blocks, 256, 0, st>>>(*a);
    else gated_norm_kernel<float, true><<<blocks, 256, 0, st>>>(*a);
  } else {
    const int threads = std::min(512, (a->group_size / 4 + 31) / 32 * 32);
    if (a->dtype == NX_BF16) gated_norm_kernel<__nv_bfloat16, false><<<static_cast<int>(items), threads, 0, st>>>(*a);
    else gated_norm_kernel<float, false><<<static_cast<int>(items), threads, 0, st>>>(*a);
  }
  return launch_status();
}

extern "C" int nx_token_side_gate(const float* a, int64_t lda, const int32_t* tokens, const void* table, int64_t ld_table,
                                  int offset, void* out, int64_t ldo, int rows, int dim, int dtype, nx_stream_t stream) {
  if (dim <= 0 || ldo < dim) return -1;
  if (rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int tx = std::max(32, std::min(128, static_cast<int>((ldo + 31) / 32 * 32))), ty = rows >= 1024 ? 512 / tx : 1;
  const dim3 threads(tx, ty);
  const int blocks = (rows + ty - 1) / ty;
  if (dtype == NX_BF16)
    token_side_kernel<__nv_bfloat16><<<blocks, threads, 0, st>>>(a, lda, tokens, (const __nv_bfloat16*)table,
                                                               ld_table, offset, (__nv_bfloat16*)out, ldo, dim, rows);
  else if (dtype == NX_F32)
    token_side_kernel<float><<<blocks, threads, 0, st>>>(a, lda, tokens, (const float*)table, ld_table, offset,
                                                       (float*)out, ldo, dim, rows);
  else
    return -1;
  return launch_status();
}

extern "C" int nx_glu(const void* h, int64_t ldh, void* out, int64_t ldo, int rows, int half, int interleaved, NxGlu glu,
                      int dtype, nx_stream_t stream) {
  if (half <= 0 || glu.kind < NX_GLU_SILU || glu.kind > NX_GLU_CLAMP || (interleaved && half % 8)) return -1;
  if (rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = half % 8 == 0 && ldh % 8 == 0 && ldo % 8 == 0 &&
                   ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  for (int r0 = 0; r0 < rows; r0 += 65535) {
    const int n = std::min(65535, rows - r0);
    dim3 grid((half / (vec ? 8 : 1) + 127) / 128, n);
#define NX_SM(T_, V_) \
  glu_kernel<T_, V_><<<grid, 128, 0, st>>>((const T_*)h + r0 * ldh, ldh, (T_*)out + r0 * ldo, ldo, half, interleaved, glu)
    if (dtype == NX_BF16) { if (vec) NX_SM(__nv_bfloat16, 8); else NX_SM(__nv_bfloat16, 1); }
    else if (dtype == NX_F32) { if (vec) NX_SM(float, 8); else NX_SM(float, 1); }
    else return -1;
#undef NX_SM
  }
  return launch_status();
}

extern "C" int nx_silu_mul(const void* h, int64_t ldh, void* out, int64_t ldo, int rows, int half, int dtype,
                           nx_stream_t stream) {
  return nx_glu(h, ldh, out, ldo, rows, half, 0, NxGlu{NX_GLU_SILU, 0.0f, 0.0f, 0.0f}, dtype, stream);
}

extern "C" int nx_softcap(float* x, int64_t ld, int rows, int cols, float cap, float scale, nx_stream_t stream) {
  if (cap < 0.0f || rows > 65535) return -1;
  if (rows <= 0 || cols <= 0) return 0;
  dim3 grid((cols + 255) / 256, rows);
  softcap_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(x, ld, cols, cap, scale);
  return launch_status();
}
