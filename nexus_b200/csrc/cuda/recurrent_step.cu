// Token-by-token forms of the recurrences (see nx_api_mixers.h): Mamba-2 state-space duality, the gated delta rule and gated
// linear attention.  A block owns one tile of value columns of one head of one segment: the columns of the state are independent of
// one another, so the tile is staged in shared memory once, every token of the segment is applied to it in FP32, and it
// is written back.  This is the decode path (one token: the kernel streams the state once each way), the path of short
// prompt portions, and the FP32 path of any length.
#include "mixer_common.cuh"
#include "nx_api_mixers.h"

#include <algorithm>

namespace {
using namespace nx;

constexpr int kStepThreads = 256;

// state tile [rows][width] of a [rows][pitch] matrix, global <-> shared
__device__ __forceinline__ void load_state(float* s, const float* g, int rows, int width, int pitch, bool vec, bool zero) {
  if (zero) {
    for (int i = threadIdx.x; i < rows * width; i += blockDim.x) s[i] = 0.0f;
  } else if (vec) {
    const int w4 = width / 4;
    for (int i = threadIdx.x; i < rows * w4; i += blockDim.x)
      cp_async16(s + (i / w4) * width + (i % w4) * 4, g + static_cast<int64_t>(i / w4) * pitch + (i % w4) * 4);
    cp_async_commit();
  } else {
    for (int i = threadIdx.x; i < rows * width; i += blockDim.x) s[i] = g[static_cast<int64_t>(i / width) * pitch + i % width];
  }
}
__device__ __forceinline__ void store_state(const float* s, float* g, int rows, int width, int pitch, bool vec) {
  if (vec) {
    const int w4 = width / 4;
    for (int i = threadIdx.x; i < rows * w4; i += blockDim.x)
      *reinterpret_cast<float4*>(g + static_cast<int64_t>(i / w4) * pitch + (i % w4) * 4) =
          *reinterpret_cast<const float4*>(s + (i / w4) * width + (i % w4) * 4);
  } else {
    for (int i = threadIdx.x; i < rows * width; i += blockDim.x) g[static_cast<int64_t>(i / width) * pitch + i % width] = s[i];
  }
}

// grid (heads, column tiles, segments); shared: state [N][tile] | B [N] | C [N] | partial sums [groups of rows][tile]
template <typename T>
__global__ void __launch_bounds__(kStepThreads) ssd_step_kernel(const NxSsdArgs a, int tile) {
  extern __shared__ __align__(16) float smem[];
  const int h = blockIdx.x, p0 = blockIdx.y * tile, sg = blockIdx.z;
  const int len = a.seg.len[sg];
  if (len <= 0) return;
  const int N = a.n_state, P = a.vdim, width = min(tile, P - p0);
  const int inner = a.heads * P, g = h / (a.heads / a.groups);
  float* sS = smem;
  float* sB = sS + N * tile;
  float* sC = sB + N;
  float* sR = sC + N;
  const int ng = kStepThreads / width;                 // row groups that share a column
  const int tx = threadIdx.x % width, ty = threadIdx.x / width;
  const bool active = ty < ng;
  const bool vec = (P & 3) == 0 && (width & 3) == 0 && (p0 & 3) == 0;
  float* gS = a.state + ((static_cast<int64_t>(a.seg.seq[sg]) * a.heads + h) * N) * P + p0;
  const bool zero = a.seg.pos[sg] == 0;
  load_state(sS, gS, N, width, P, vec, zero);
  const int64_t row0 = a.seg.row0[sg];
  const T* xbc = static_cast<const T*>(a.xbc) + row0 * a.ld_xbc;
  const T* dtp = static_cast<const T*>(a.dt) + row0 * a.ld_dt + h;
  T* y = static_cast<T*>(a.y) + row0 * a.ldy + static_cast<int64_t>(h) * P + p0;
  const float rate = -expf(a.a_log[h]), dtb = a.dt_bias[h], skip = a.d_skip[h];
  if (vec && !zero) cp_async_wait<0>();
  for (int t = 0; t < len; ++t, xbc += a.ld_xbc, dtp += a.ld_dt, y += a.ldy) {
    for (int n = threadIdx.x; n < N; n += kStepThreads) {
      sB[n] = Num<T>::load(xbc + inner + g * N + n);
      sC[n] = Num<T>::load(xbc + inner + (a.groups + g) * N + n);
    }
    const float x = active ? Num<T>::load(xbc + h * P + p0 + tx) : 0.0f;
    const float dt = softplus_exact(Num<T>::load(dtp) + dtb);
    const float decay = expf(rate * dt), dx = dt * x;
    __syncthreads();
    float acc = 0.0f;
    if (active) {
#pragma unroll 4
      for (int n = ty; n < N; n += ng) {
        const float s = sS[n * width + tx] * decay + sB[n] * dx;
        sS[n * width + tx] = s;
        acc += s * sC[n];
      }
      sR[ty * width + tx] = acc;
    }
    __syncthreads();
    if (ty == 0) {
      for (int i = 1; i < ng; ++i) acc += sR[i * width + tx];
      Num<T>::store(y + tx, acc + skip * x);
    }
  }
  __syncthreads();
  store_state(sS, gS, N, width, P, vec);
}

// grid (heads, column tiles, segments); shared: state [D][tile] | k [D] | q [D] | partial sums [2][row groups][tile]
template <typename T>
__global__ void __launch_bounds__(kStepThreads) delta_step_kernel(const NxDeltaArgs a, int tile) {
  extern __shared__ __align__(16) float smem[];
  const int h = blockIdx.x, v0 = blockIdx.y * tile, sg = blockIdx.z;
  const int len = a.seg.len[sg];
  if (len <= 0) return;
  const int D = a.dim, Dv = a.vdim, width = min(tile, Dv - v0);
  const int hk = h / (a.heads / a.kv_heads), kcols = a.kv_heads * D;
  float* sS = smem;
  float* sK = sS + D * tile;
  float* sQ = sK + D;
  float* sR = sQ + D;
  const int ng = kStepThreads / width;
  const int tx = threadIdx.x % width, ty = threadIdx.x / width, lane = threadIdx.x & 31;
  const bool active = ty < ng;
  const bool vec = (Dv & 3) == 0 && (width & 3) == 0 && (v0 & 3) == 0;
  float* gS = a.state + ((static_cast<int64_t>(a.seg.seq[sg]) * a.heads + h) * D) * Dv + v0;
  const bool zero = a.seg.pos[sg] == 0;
  load_state(sS, gS, D, width, Dv, vec, zero);
  const int64_t row0 = a.seg.row0[sg];
  const T* qkv = static_cast<const T*>(a.qkv) + row0 * a.ld_qkv;
  const T* bp = static_cast<const T*>(a.b) + row0 * a.ld_ba + h;
  const T* ap = static_cast<const T*>(a.a) + row0 * a.ld_ba + h;
  T* o = static_cast<T*>(a.o) + row0 * a.ldo + static_cast<int64_t>(h) * Dv + v0;
  const float rate = -expf(a.a_log[h]), dtb = a.dt_bias[h];
  float* sR2 = sR + ng * width;
  if (vec && !zero) cp_async_wait<0>();
  for (int t = 0; t < len; ++t, qkv += a.ld_qkv, bp += a.ld_ba, ap += a.ld_ba, o += a.ldo) {
    // every warp forms the three sums over the head dimension by itself
    float qq = 0.0f, kk = 0.0f, qk = 0.0f;
    for (int d = lane; d < D; d += 32) {
      const float q = Num<T>::load(qkv + hk * D + d), k = Num<T>::load(qkv + kcols + hk * D + d);
      if (threadIdx.x < 32) {
        sQ[d] = q;
        sK[d] = k;
      }
      qq += q * q;
      kk += k * k;
      qk += q * k;
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    qk = warp_sum(qk);
    const float rq = a.q_scale / sqrtf(qq + a.unit_eps), rk = 1.0f / sqrtf(kk + a.unit_eps);
    const float beta = sigmoid_exact(Num<T>::load(bp));
    const float gate = expf(rate * softplus_exact(Num<T>::load(ap) + dtb));
    const float v = active ? Num<T>::load(qkv + 2 * kcols + h * Dv + v0 + tx) : 0.0f;
    __syncthreads();
    float sk = 0.0f, sq = 0.0f;
    if (active) {
#pragma unroll 4
      for (int d = ty; d < D; d += ng) {
        const float s = sS[d * width + tx];
        sk += s * sK[d];
        sq += s * sQ[d];
      }
      sR[ty * width + tx] = sk;
      sR2[ty * width + tx] = sq;
    }
    __syncthreads();
    if (active) {
      sk = sq = 0.0f;
      for (int i = 0; i < ng; ++i) {
        sk += sR[i * width + tx];
        sq += sR2[i * width + tx];
      }
      const float u = beta * (v - gate * rk * sk);
      if (ty == 0) Num<T>::store(o + tx, gate * rq * sq + rq * rk * qk * u);
      const float ku = rk * u;
#pragma unroll 4
      for (int d = ty; d < D; d += ng) sS[d * width + tx] = gate * sS[d * width + tx] + sK[d] * ku;
    }
    __syncthreads();
  }
  store_state(sS, gS, D, width, Dv, vec);
}

// grid (heads, column tiles, segments); shared: state [D][tile] | k [D] | q [D] | decay [D] | partial sums [row groups][tile]
template <typename T>
__global__ void __launch_bounds__(kStepThreads) gla_step_kernel(const NxGlaArgs a, int tile) {
  extern __shared__ __align__(16) float smem[];
  const int h = blockIdx.x, v0 = blockIdx.y * tile, sg = blockIdx.z;
  const int len = a.seg.len[sg];
  if (len <= 0) return;
  const int D = a.dim, Dv = a.vdim, width = min(tile, Dv - v0);
  float* sS = smem;
  float* sK = sS + D * tile;
  float* sQ = sK + D;
  float* sA = sQ + D;
  float* sR = sA + D;
  const int ng = kStepThreads / width;
  const int tx = threadIdx.x % width, ty = threadIdx.x / width;
  const bool active = ty < ng;
  const bool vec = (Dv & 3) == 0 && (width & 3) == 0 && (v0 & 3) == 0;
  float* gS = a.state + ((static_cast<int64_t>(a.seg.seq[sg]) * a.heads + h) * D) * Dv + v0;
  const bool zero = a.seg.pos[sg] == 0;
  load_state(sS, gS, D, width, Dv, vec, zero);
  const int64_t row0 = a.seg.row0[sg];
  const T* q = static_cast<const T*>(a.q) + row0 * a.ld + static_cast<int64_t>(h) * D;
  const T* k = static_cast<const T*>(a.k) + row0 * a.ld + static_cast<int64_t>(h) * D;
  const T* v = static_cast<const T*>(a.v) + row0 * a.ld + static_cast<int64_t>(h) * Dv + v0;
  const float* dec = a.decay + row0 * a.ld_decay + static_cast<int64_t>(h) * D;
  T* o = static_cast<T*>(a.o) + row0 * a.ldo + static_cast<int64_t>(h) * Dv + v0;
  if (vec && !zero) cp_async_wait<0>();
  for (int t = 0; t < len; ++t, q += a.ld, k += a.ld, v += a.ld, dec += a.ld_decay, o += a.ldo) {
    for (int d = threadIdx.x; d < D; d += kStepThreads) {
      sK[d] = Num<T>::load(k + d);
      sQ[d] = a.q_scale * Num<T>::load(q + d);
      sA[d] = exp2f(dec[d]);
    }
    const float x = active ? Num<T>::load(v + tx) : 0.0f;
    __syncthreads();
    float acc = 0.0f;
    if (active) {
#pragma unroll 4
      for (int d = ty; d < D; d += ng) {
        const float s = sS[d * width + tx] * sA[d] + sK[d] * x;
        sS[d * width + tx] = s;
        acc += s * sQ[d];
      }
      sR[ty * width + tx] = acc;
    }
    __syncthreads();
    if (ty == 0) {
      for (int i = 1; i < ng; ++i) acc += sR[i * width + tx];
      Num<T>::store(o + tx, acc);
    }
  }
  __syncthreads();
  store_state(sS, gS, D, width, Dv, vec);
}

int pick_tile(int cols, int rows, size_t extra_bytes) {
  // a tile of 32 columns keeps many blocks resident; wider only for wide heads of few rows
  int tile = std::min(cols, 32);
  while (tile > 1 && static_cast<size_t>(rows) * tile * 4 + extra_bytes > 200 * 1024) tile = (tile + 1) / 2;
  return tile;
}

template <typename K>
int set_smem(K kernel, size_t bytes) {
  if (bytes <= 48 * 1024) return 0;
  return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)) == cudaSuccess ? 0 : -2;
}

}  // namespace

extern "C" int nx_ssd_step(const NxSsdArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->heads <= 0 || a->groups <= 0 || a->heads % a->groups || a->n_state <= 0 || a->vdim <= 0) return -1;
  if (a->seg.count <= 0) return 0;
  if (a->seg.count > 65535) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int tile = pick_tile(a->vdim, a->n_state, static_cast<size_t>(2 * a->n_state + kStepThreads) * 4);
  const size_t smem = (static_cast<size_t>(a->n_state) * tile + 2 * a->n_state + kStepThreads) * sizeof(float);
  if (smem > 220 * 1024) return -1;
  dim3 grid(a->heads, (a->vdim + tile - 1) / tile, a->seg.count);
  if (a->dtype == NX_BF16) {
    if (set_smem(ssd_step_kernel<__nv_bfloat16>, smem)) return -2;
    ssd_step_kernel<__nv_bfloat16><<<grid, kStepThreads, smem, st>>>(*a, tile);
  } else if (a->dtype == NX_F32) {
    if (set_smem(ssd_step_kernel<float>, smem)) return -2;
    ssd_step_kernel<float><<<grid, kStepThreads, smem, st>>>(*a, tile);
  } else {
    return -1;
  }
  return launch_status();
}

extern "C" int nx_delta_step(const NxDeltaArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0) return -1;
  if (a->seg.count <= 0) return 0;
  if (a->seg.count > 65535) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int tile = pick_tile(a->vdim, a->dim, static_cast<size_t>(2 * a->dim + 2 * kStepThreads) * 4);
  const size_t smem = (static_cast<size_t>(a->dim) * tile + 2 * a->dim + 2 * kStepThreads) * sizeof(float);
  if (smem > 220 * 1024) return -1;
  dim3 grid(a->heads, (a->vdim + tile - 1) / tile, a->seg.count);
  if (a->dtype == NX_BF16) {
    if (set_smem(delta_step_kernel<__nv_bfloat16>, smem)) return -2;
    delta_step_kernel<__nv_bfloat16><<<grid, kStepThreads, smem, st>>>(*a, tile);
  } else if (a->dtype == NX_F32) {
    if (set_smem(delta_step_kernel<float>, smem)) return -2;
    delta_step_kernel<float><<<grid, kStepThreads, smem, st>>>(*a, tile);
  } else {
    return -1;
  }
  return launch_status();
}

extern "C" int nx_gla_step(const NxGlaArgs* a, nx_stream_t stream) {
  if (a == nullptr || a->heads <= 0 || a->dim <= 0 || a->vdim <= 0) return -1;
  if (a->seg.count <= 0) return 0;
  if (a->seg.count > 65535) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int tile = pick_tile(a->vdim, a->dim, static_cast<size_t>(3 * a->dim + kStepThreads) * 4);
  const size_t smem = (static_cast<size_t>(a->dim) * tile + 3 * a->dim + kStepThreads) * sizeof(float);
  if (smem > 220 * 1024) return -1;
  dim3 grid(a->heads, (a->vdim + tile - 1) / tile, a->seg.count);
  if (a->dtype == NX_BF16) {
    if (set_smem(gla_step_kernel<__nv_bfloat16>, smem)) return -2;
    gla_step_kernel<__nv_bfloat16><<<grid, kStepThreads, smem, st>>>(*a, tile);
  } else if (a->dtype == NX_F32) {
    if (set_smem(gla_step_kernel<float>, smem)) return -2;
    gla_step_kernel<float><<<grid, kStepThreads, smem, st>>>(*a, tile);
  } else {
    return -1;
  }
  return launch_status();
}
