// Pieces the tcgen05 attention kernels share: descriptors of swizzled tiles, the MMA that reads its A operand from TMEM,
// constants of the online softmax.
#pragma once
#include "sm100_ptx.cuh"

namespace nx {

constexpr float kLog2e = 1.4426950408889634f;
constexpr float kRescaleStep = 8.0f;  // log2 of the growth of the row maximum that forces a rescale of the output tile

// K-major operand: address of k-step `ks` (16 elements) in a tile of HD/64 (or cols/64) slabs of `rows` rows.
__device__ __forceinline__ uint64_t desc_kmajor(uint32_t tile_addr, int rows, int ks) {
  const uint32_t a = tile_addr + static_cast<uint32_t>((ks >> 2) * rows * 128 + (ks & 3) * 32);
  return make_smem_desc_sw128(a, 16, 1024);
}
// MN-major view of a [k_rows][mn] tile stored as mn/64 slabs of [k_rows][64]: k-step `ks` = 16 rows.
__device__ __forceinline__ uint64_t desc_mnmajor(uint32_t tile_addr, int k_rows, int ks) {
  const uint32_t a = tile_addr + static_cast<uint32_t>(ks * 2048);
  return make_smem_desc_sw128(a, static_cast<uint32_t>(k_rows * 128), 1024);
}

// what k-step `ks` adds to the address field (bytes >> 4) of a K-major / MN-major descriptor built for k-step 0
__device__ __forceinline__ uint64_t kstep_kmajor(int rows, int ks) {
  return static_cast<uint64_t>((ks >> 2) * rows * 8 + (ks & 3) * 2);
}
__device__ __forceinline__ uint64_t kstep_mnmajor(int ks) { return static_cast<uint64_t>(ks * 128); }

__device__ __forceinline__ float ex2f(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// D[tmem] (+)= A[tmem] * B[smem]: the A operand (128 rows on the lanes, two BF16 per column along K) is read from TMEM
__device__ __forceinline__ void umma_f16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc,
                                            uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t"
      "}" ::"r"(tmem_d),
      "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
      : "memory");
}

}  // namespace nx
