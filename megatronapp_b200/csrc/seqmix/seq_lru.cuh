// The element functions of the real-gated linear recurrent unit, shared by its kernels.
#pragma once
#include <math.h>

#include "seq_common.cuh"

namespace b200seq {
namespace dev {

constexpr int kLruRun = 64;                                // tokens of a sequence that one thread walks

__device__ __forceinline__ float softplusf_(float z) { return z > 30.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float gelu_tanhf_(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z)));
}
// decay a = exp(-rate * r) and what a token writes, sqrt(1 - a^2) * i * u, from the gates' pre-activations
__device__ __forceinline__ void lru_gates(float r_pre, float i_pre, float u, float rate, float* a, float* put) {
  const float la = -rate * sigmoidf_(r_pre);
  *a = expf(la);
  *put = sqrtf(-expm1f(2.f * la)) * sigmoidf_(i_pre) * u;
}

}  // namespace dev
}  // namespace b200seq
