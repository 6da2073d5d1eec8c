// Helpers shared by the mixer kernels: vector loads of any dtype as FP32, the activations in full FP32 accuracy, and the
// warp-level BF16 tensor-core tile (m16n8k16) with its shared-memory fragment loads.
#pragma once
#include "common.cuh"
#include "glu.cuh"
#include "nx_api_mixers.h"

namespace nx {

template <typename T, int V>
__device__ __forceinline__ void load_vec(const T* p, float (&v)[V]) {
  if constexpr (V == 1) {
    v[0] = Num<T>::load(p);
  } else {
    constexpr int kBytes = V * static_cast<int>(sizeof(T));
    alignas(16) T buf[V];
    if constexpr (kBytes % 16 == 0) {
#pragma unroll
      for (int i = 0; i < kBytes / 16; ++i) reinterpret_cast<uint4*>(buf)[i] = reinterpret_cast<const uint4*>(p)[i];
    } else if constexpr (kBytes == 8) {
      *reinterpret_cast<uint2*>(buf) = *reinterpret_cast<const uint2*>(p);
    } else {
      *reinterpret_cast<uint32_t*>(buf) = *reinterpret_cast<const uint32_t*>(p);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = Num<T>::load(buf + i);
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_vec(T* p, const float (&v)[V]) {
  if constexpr (V == 1) {
    Num<T>::store(p, v[0]);
  } else {
    constexpr int kBytes = V * static_cast<int>(sizeof(T));
    alignas(16) T buf[V];
#pragma unroll
    for (int i = 0; i < V; ++i) Num<T>::store(buf + i, v[i]);
    if constexpr (kBytes % 16 == 0) {
#pragma unroll
      for (int i = 0; i < kBytes / 16; ++i) reinterpret_cast<uint4*>(p)[i] = reinterpret_cast<const uint4*>(buf)[i];
    } else if constexpr (kBytes == 8) {
      *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(buf);
    } else {
      *reinterpret_cast<uint32_t*>(p) = *reinterpret_cast<const uint32_t*>(buf);
    }
  }
}

__device__ __forceinline__ float silu_exact(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_exact(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

// the hardware exponential and reciprocal (results below the normal range flush to zero)
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// ---- BF16 tensor-core fragments -----------------------------------------------------------------
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two floats as one BF16 pair, and what the rounding left over as a second pair (hi + lo keeps 16 bits of mantissa)
__device__ __forceinline__ uint32_t bf16_pair(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ void bf16_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  hi = *reinterpret_cast<const uint32_t*>(&v);
  lo = bf16_pair(a - __low2float(v), b - __high2float(v));
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

}  // namespace nx
