// Gated activations of a gate and a value (NxGlu).
#pragma once
#include <math.h>

#include "nx_api.h"

namespace nx {

__device__ __forceinline__ float sigmoid_exact(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float gelu_tanh_exact(float x) {
  return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
}

// kExact: full FP32 accuracy, else the fast exponential and division (for results that are rounded to BF16)
template <bool kExact>
__device__ __forceinline__ float sigmoid_as(float x) {
  return kExact ? sigmoid_exact(x) : __fdividef(1.0f, 1.0f + __expf(-x));
}
template <bool kExact>
__device__ __forceinline__ float glu_apply(const NxGlu& f, float g, float u) {
  if (f.kind == NX_GLU_SILU) return g * sigmoid_as<kExact>(g) * u;
  if (f.kind == NX_GLU_GELU)          // (1 + tanh z) / 2 = sigmoid(2 z)
    return (kExact ? gelu_tanh_exact(g) : g * sigmoid_as<false>(1.5957691216057308f * (g + 0.044715f * g * g * g))) * u;
  g = fminf(g, f.limit);
  u = fminf(fmaxf(u, -f.limit), f.limit);
  return g * sigmoid_as<kExact>(f.slope * g) * (u + f.offset);
}

}  // namespace nx
