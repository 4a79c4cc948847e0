// Squashing norm without row statistics, fused with the residual addition around it (sm_100a):
//
//   x <- x_scale * x + mult * N_o(a);   h = N_n(x);   N(z) = tanh(alpha z) * w + b        (alpha a scalar, w and b per channel)
//
// The stream x is fp32; addends, weights and h are `T` (float or __nv_bfloat16); all arithmetic is fp32.  Everything is element by
// element, so a thread keeps the weights of its columns in registers and walks down the rows.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>
#include <algorithm>

#include "seq_common.cuh"
#include "seqmix_api.h"

namespace b200seq {

namespace {

using namespace dev;

constexpr int kSquashThreads = 128;

template <typename T, int V> struct Row;                   // V neighbouring columns of a row as fp32
template <> struct Row<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 r = *reinterpret_cast<const float4*>(p);
    v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <> struct Row<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 r;
    r.x = *reinterpret_cast<const uint32_t*>(&a); r.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = r;
  }
};
template <typename T> struct Row<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = ld(p); }
  static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { st(p, v[0]); }
};

// grid (column chunks of kSquashThreads * V, row groups)
template <typename T, int V>
__global__ void __launch_bounds__(kSquashThreads) squash_add_kernel(SquashArgs p, int n_rows) {
  const int c = (blockIdx.x * kSquashThreads + threadIdx.x) * V;
  if (c >= p.W) return;
  const T* a = static_cast<const T*>(p.a);
  T* h = static_cast<T*>(p.h);
  const bool normed = p.wo != nullptr;
  float wo[V], bo[V], wn[V], bn[V], ao = 0.f, an = 0.f;
#pragma unroll
  for (int i = 0; i < V; ++i) { wo[i] = p.mult; bo[i] = 0.f; wn[i] = 0.f; bn[i] = 0.f; }
  if (normed) {                                            // mult * (tanh(.) w + b): the multiplier goes into the weights
    Row<T, V>::load(static_cast<const T*>(p.wo) + c, wo);
    Row<T, V>::load(static_cast<const T*>(p.bo) + c, bo);
    ao = ld(static_cast<const T*>(p.alpha_o));
#pragma unroll
    for (int i = 0; i < V; ++i) { wo[i] *= p.mult; bo[i] *= p.mult; }
  }
  if (h != nullptr) {
    Row<T, V>::load(static_cast<const T*>(p.wn) + c, wn);
    Row<T, V>::load(static_cast<const T*>(p.bn) + c, bn);
    an = ld(static_cast<const T*>(p.alpha_n));
  }
  const bool writes = a != nullptr || p.x_scale != 1.f;
  for (int t = blockIdx.y; t < n_rows; t += gridDim.y) {
    float v[V], av[V];
    float* x = p.x + static_cast<int64_t>(t) * p.W + c;
    Row<float, V>::load(x, v);
    if (a != nullptr) Row<T, V>::load(a + t * p.lda + c, av);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      v[i] *= p.x_scale;
      if (a != nullptr) v[i] = fmaf(normed ? tanhf(ao * av[i]) : av[i], wo[i], v[i] + bo[i]);
    }
    if (writes) Row<float, V>::store(x, v);
    if (h != nullptr) {
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = fmaf(tanhf(an * v[i]), wn[i], bn[i]);
      Row<T, V>::store(h + static_cast<int64_t>(t) * p.W + c, v);
    }
  }
}

template <typename T, int V>
void launch_squash(const SquashArgs& p, int n_tok, cudaStream_t s) {
  const int chunks = (p.W + kSquashThreads * V - 1) / (kSquashThreads * V);
  const int groups = std::min(n_tok, std::max(1, 148 * 16 / chunks));
  squash_add_kernel<T, V><<<dim3(chunks, std::min(groups, 65535)), kSquashThreads, 0, s>>>(p, n_tok);
}

}  // namespace

void squash_add(const SquashArgs& p, int n_tok, bool bf16, cudaStream_t s) {
  if (n_tok == 0) return;
  auto ok = [](const void* ptr, int64_t row) { return ptr == nullptr || (row % 4 == 0 && reinterpret_cast<uintptr_t>(ptr) % 16 == 0); };
  const bool vec = p.W % 4 == 0 && ok(p.x, p.W) && ok(p.a, p.lda) && ok(p.h, p.W) && ok(p.wo, 0) && ok(p.bo, 0) && ok(p.wn, 0) && ok(p.bn, 0);
  if (bf16) {
    if (vec) launch_squash<__nv_bfloat16, 4>(p, n_tok, s);
    else launch_squash<__nv_bfloat16, 1>(p, n_tok, s);
  } else {
    if (vec) launch_squash<float, 4>(p, n_tok, s);
    else launch_squash<float, 1>(p, n_tok, s);
  }
}

}  // namespace b200seq
