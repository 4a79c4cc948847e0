// Device helpers shared by the sequence-mixing kernels: typed loads / stores through fp32 and warp reductions.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace b200seq {
namespace dev {

template <typename T> __device__ __forceinline__ float ld(const T* p);
template <> __device__ __forceinline__ float ld<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ld<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void st(T* p, float v);
template <> __device__ __forceinline__ void st<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void st<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
__device__ __forceinline__ float sigmoidf_(float x) { return 1.0f / (1.0f + expf(-x)); }

// Sine and cosine of pos * rate, the rate given in full turns as the sum of two floats: the product's rounding error is carried
// along, so the fraction of a turn keeps fp32 accuracy for far positions.
__device__ __forceinline__ void turn_angle(const float* rate, int pos, float* sn, float* cs) {
  const float p = static_cast<float>(pos), hi = rate[0];
  const float prod = __fmul_rn(p, hi), err = __fmaf_rn(p, hi, -prod);
  const float frac = (prod - rintf(prod)) + __fmaf_rn(p, rate[1], err);
  sincospif(2.f * frac, sn, cs);
}

}  // namespace dev
}  // namespace b200seq
