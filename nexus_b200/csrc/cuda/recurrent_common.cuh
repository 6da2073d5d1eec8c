// What the chunked tensor-core recurrences share: tiles of a chunk in shared memory, fragment addresses, FP32 accumulators
// split into BF16 pairs.
#pragma once
#include "mixer_common.cuh"
#include "nx_api_mixers.h"

namespace nx {

constexpr int kQ = 64;                 // tokens per chunk
constexpr float kLog2e = 1.4426950408889634f;

// rows x cols BF16 of a row-major matrix into shared memory [64][LD]; rows past `rows` and columns past `cols` (up to PAD)
// are zeros.  `vec`: 16-byte copies are possible.
template <int PAD>
__device__ __forceinline__ void load_tile(__nv_bfloat16* dst, const __nv_bfloat16* src, int64_t ld, int rows, int cols, bool vec) {
  constexpr int LD = PAD + 8, CH = PAD / 8;
  for (int i = threadIdx.x; i < kQ * CH; i += blockDim.x) {
    const int r = i / CH, c = (i % CH) * 8;
    __nv_bfloat16* d = dst + r * LD + c;
    if (r < rows && c < cols) {
      const __nv_bfloat16* s = src + r * ld + c;
      if (vec) {
        cp_async16(d, s);
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) d[e] = c + e < cols ? s[e] : __float2bfloat16_rn(0.0f);
      }
    } else {
      *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
    }
  }
}

// fragment addresses inside a [rows][LD] BF16 tile
template <int LD>
__device__ __forceinline__ uint32_t addr_a(const __nv_bfloat16* t, int row, int col) {       // A, row-major
  const int lane = threadIdx.x & 31;
  return smem_addr(t + (row + (lane & 15)) * LD + col + (lane >> 4) * 8);
}
template <int LD>
__device__ __forceinline__ uint32_t addr_a_t(const __nv_bfloat16* t, int k, int m) {         // A = transpose of the tile
  const int lane = threadIdx.x & 31;
  return smem_addr(t + (k + ((lane >> 4) << 3) + (lane & 7)) * LD + m + ((lane >> 3) & 1) * 8);
}
template <int LD>
__device__ __forceinline__ uint32_t addr_b(const __nv_bfloat16* t, int n, int k) {           // B[k][n] = tile[n][k]
  const int lane = threadIdx.x & 31;
  return smem_addr(t + (n + (lane & 7) + ((lane >> 4) << 3)) * LD + k + ((lane >> 3) & 1) * 8);
}
template <int LD>
__device__ __forceinline__ uint32_t addr_b_t(const __nv_bfloat16* t, int k, int n) {         // B[k][n] = tile[k][n]
  const int lane = threadIdx.x & 31;
  return smem_addr(t + (k + (lane & 15)) * LD + n + (lane >> 4) * 8);
}

template <int N>
__device__ __forceinline__ void zero(float (&d)[N][4]) {
#pragma unroll
  for (int i = 0; i < N; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) d[i][e] = 0.0f;
}

// an FP32 accumulator tile (16 rows x 8 NT columns) as a pair of BF16 tiles in shared memory
template <int NT, int LD>
__device__ __forceinline__ void store_split(__nv_bfloat16* hi, __nv_bfloat16* lo, int row, const float (&v)[NT][4]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      uint32_t h, l;
      bf16_split(v[n][2 * i], v[n][2 * i + 1], h, l);
      const int o = (row + i * 8 + (lane >> 2)) * LD + n * 8 + (lane & 3) * 2;
      *reinterpret_cast<uint32_t*>(hi + o) = h;
      *reinterpret_cast<uint32_t*>(lo + o) = l;
    }
}

}  // namespace nx
