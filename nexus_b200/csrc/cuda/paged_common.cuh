// What the attention kernels over a paged cache share: the tile lookup in a segment table and page arithmetic.
#pragma once
#include "common.cuh"
#include "nx_api_mixers.h"

namespace nx {

// which segment, and which tile of `per` tokens inside it, flat tile index `tile` is; executed by one full warp
__device__ __forceinline__ bool find_tile(const NxSegments& s, int per, int tile, int& seg, int& off) {
  const int lane = threadIdx.x & 31;
  int base = 0;
  for (int i0 = 0; i0 < s.count; i0 += 32) {
    const int i = i0 + lane;
    const int n = i < s.count ? (s.len[i] + per - 1) / per : 0;
    int incl = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += v;
    }
    const unsigned hit = __ballot_sync(0xffffffffu, base + incl > tile);
    if (hit) {
      const int first = __ffs(hit) - 1;
      seg = i0 + first;
      off = tile - base - __shfl_sync(0xffffffffu, incl - n, first);
      return true;
    }
    base += __shfl_sync(0xffffffffu, incl, 31);
  }
  return false;
}

__device__ __forceinline__ int log2_of(int n) { return (n & (n - 1)) == 0 ? 31 - __clz(n) : -1; }

// cache slot of position j; shift: log2 of a power-of-two block size, else -1
__device__ __forceinline__ int64_t page_slot(const int32_t* table, int block_size, int shift, int j) {
  if (shift >= 0) return (static_cast<int64_t>(table[j >> shift]) << shift) + (j & (block_size - 1));
  return static_cast<int64_t>(table[j / block_size]) * block_size + j % block_size;
}

}  // namespace nx
