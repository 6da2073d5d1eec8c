// Residual of several streams (see nx_api_mixers.h): every sublayer reads a weighted sum of the streams and writes to a mixture of
// all of them.  One kernel per sublayer: the old streams are read once, mixed with the sublayer's output, written, and the next
// sublayer's normed input is formed on the way.  One block per row, everything in FP32.
#include "common.cuh"
#include "mixer_common.cuh"
#include "nx_api_mixers.h"

#include <algorithm>

namespace {
using namespace nx;

constexpr int kMaxThreads = 256;

// S: streams the registers hold (a.streams <= S)
template <typename T, int V, int S>
__global__ void __launch_bounds__(kMaxThreads) stream_residual_kernel(const NxStreamResidualArgs a) {
  extern __shared__ __align__(16) float s_u[];          // [cols]: the weighted sum of the streams
  __shared__ float s_red[32], s_mix[S * S], s_out[S], s_in[S];
  const int64_t r = blockIdx.x;
  const int cols = a.cols, n = a.streams;
  float* xr = a.x + r * n * cols;
  const bool embed = a.table != nullptr, add = !embed && a.y != nullptr;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) {
    const int s = i / S, t = i % S;
    s_mix[i] = add && s < n && t < n ? a.mix[s * n + t] : 0.0f;
    if (i < S) {
      s_out[i] = add && i < n ? a.out[i] : 0.0f;
      s_in[i] = i < n ? (a.in != nullptr ? a.in[i] : 1.0f) : 0.0f;
    }
  }
  __syncthreads();
  float mix[S][S], out[S], in[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    out[s] = s_out[s];
    in[s] = s_in[s];
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = s_mix[s * S + t];
  }
  float ss = 0.0f;
  for (int c = threadIdx.x * V; c < cols; c += blockDim.x * V) {
    float u[V];
#pragma unroll
    for (int j = 0; j < V; ++j) u[j] = 0.0f;
    if (embed) {
      float e[V], total = 0.0f;
      load_vec<T, V>(static_cast<const T*>(a.table) + static_cast<int64_t>(a.tokens[r]) * cols + c, e);
      if (a.pos_table != nullptr) {
        float p[V];
        load_vec<T, V>(static_cast<const T*>(a.pos_table) + static_cast<int64_t>(a.positions[r]) * cols + c, p);
#pragma unroll
        for (int j = 0; j < V; ++j) e[j] = e[j] * a.embed_scale + p[j];
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) e[j] *= a.embed_scale;
      }
#pragma unroll
      for (int s = 0; s < S; ++s) {
        total += in[s];
        if (s < n) store_vec<float, V>(xr + static_cast<int64_t>(s) * cols + c, e);
      }
#pragma unroll
      for (int j = 0; j < V; ++j) u[j] = total * e[j];
    } else {
      float x[S][V], y[V];
#pragma unroll
      for (int s = 0; s < S; ++s) {
        if (s < n) {
          load_vec<float, V>(xr + static_cast<int64_t>(s) * cols + c, x[s]);
        } else {
#pragma unroll
          for (int j = 0; j < V; ++j) x[s][j] = 0.0f;
        }
      }
      if (add) {
        load_vec<T, V>(static_cast<const T*>(a.y) + r * a.ldy + c, y);
#pragma unroll
        for (int t = 0; t < S; ++t) {
          if (t >= n) continue;
          float v[V];
#pragma unroll
          for (int j = 0; j < V; ++j) {
            v[j] = out[t] * y[j];
#pragma unroll
            for (int s = 0; s < S; ++s) v[j] += mix[s][t] * x[s][j];
            u[j] += in[t] * v[j];
          }
          store_vec<float, V>(xr + static_cast<int64_t>(t) * cols + c, v);
        }
      } else {
#pragma unroll
        for (int s = 0; s < S; ++s)
#pragma unroll
          for (int j = 0; j < V; ++j) u[j] += in[s] * x[s][j];
      }
    }
    store_vec<float, V>(s_u + c, u);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += u[j] * u[j];
  }
  if (a.h == nullptr) return;
  const float inv = 1.0f / sqrtf(block_sum(ss, s_red) / static_cast<float>(cols) + a.eps);
  T* o = static_cast<T*>(a.h) + r * a.ldh;
  for (int c = threadIdx.x * V; c < cols; c += blockDim.x * V) {   // each thread re-reads its own columns
    float v[V], w[V];
    load_vec<float, V>(s_u + c, v);
    load_vec<float, V>(a.w_next + c, w);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] *= inv * w[j];
    store_vec<T, V>(o + c, v);
  }
  for (int c = cols + threadIdx.x; c < a.ldh; c += blockDim.x) Num<T>::store(o + c, 0.0f);
}

template <typename T, int V>
int launch(const NxStreamResidualArgs* a, cudaStream_t st) {
  const int threads = std::max(64, std::min(kMaxThreads, (a->cols / V + 31) / 32 * 32));
  const size_t smem = static_cast<size_t>(a->cols) * sizeof(float);
  const auto run = [&](auto kernel) {
    if (smem > 40 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
      return -2;
    kernel<<<a->rows, threads, smem, st>>>(*a);
    return launch_status();
  };
  if (a->streams <= 2) return run(stream_residual_kernel<T, V, 2>);
  if (a->streams <= 3) return run(stream_residual_kernel<T, V, 3>);
  if (a->streams <= 4) return run(stream_residual_kernel<T, V, 4>);
  return run(stream_residual_kernel<T, V, 8>);
}

}  // namespace

extern "C" int nx_stream_residual(const NxStreamResidualArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->x == nullptr || a->cols <= 0 || a->cols > 49152 || a->streams < 1 || a->streams > 8) return -1;
  if (a->table != nullptr && (a->tokens == nullptr || (a->pos_table != nullptr && a->positions == nullptr))) return -1;
  if (a->table == nullptr && a->y != nullptr && (a->mix == nullptr || a->out == nullptr || a->ldy < a->cols)) return -1;
  if (a->h != nullptr && (a->w_next == nullptr || a->ldh < a->cols)) return -1;
  if (a->rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = a->cols % 4 == 0 && a->ldy % 4 == 0 && a->ldh % 4 == 0 && al(a->x) && al(a->table) && al(a->pos_table) && al(a->y) &&
                   al(a->h) && al(a->w_next);
  if (a->dtype == NX_BF16) return vec ? launch<__nv_bfloat16, 4>(a, st) : launch<__nv_bfloat16, 1>(a, st);
  if (a->dtype == NX_F32) return vec ? launch<float, 4>(a, st) : launch<float, 1>(a, st);
  return -1;
}
