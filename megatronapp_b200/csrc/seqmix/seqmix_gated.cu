// Kernels around gated, normed sublayers with rotary heads (sm_100a): the gated addition of two sublayers fused with the norm of
// what follows, rotation / norm of whole heads written to their consumers' buffers and cache pages, the operands of a rotary
// latent attention's prompts, and a scalar gate per head.
//
// Conventions as in seqmix.cu: activations are `T` (float or __nv_bfloat16); gates, sums, statistics and angles are fp32.
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

#define SEQ_DISPATCH_T(is_bf16, ...)                      \
  if (is_bf16) { using T = __nv_bfloat16; __VA_ARGS__; }  \
  else { using T = float; __VA_ARGS__; }

// every thread gets the sum; red holds >= 32 floats and is free again after the call
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < (blockDim.x >> 5); ++i) tot += red[i];
  return tot;
}

template <typename T> __device__ __forceinline__ float4 ld4(const T* p);
template <> __device__ __forceinline__ float4 ld4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 ld4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T> __device__ __forceinline__ void st4(T* p, float4 v);
template <> __device__ __forceinline__ void st4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void st4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<const uint32_t*>(&a); raw.y = *reinterpret_cast<const uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = raw;
}

// ---------------------------------------------------------------------------------------------------------------------
// x += sigmoid(ga + ba) * a + sigmoid(gb + bb) * b;  n = (x - mean) / sqrt(var + eps) (or x / rms);  h1 = n * w1, h2 = n * w2.
// One CTA per row.  Four columns per thread and step, the row in registers; or any width through shared memory.
// ---------------------------------------------------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ void gated_add4(float4& v, const T* a, const T* g, const T* bias, int c) {
  if (a == nullptr) return;
  const float4 av = ld4(a + c);
  if (g == nullptr) { v.x += av.x; v.y += av.y; v.z += av.z; v.w += av.w; return; }
  float4 gv = ld4(g + c);
  if (bias != nullptr) { const float4 bv = ld4(bias + c); gv.x += bv.x; gv.y += bv.y; gv.z += bv.z; gv.w += bv.w; }
  v.x = fmaf(sigmoidf_(gv.x), av.x, v.x); v.y = fmaf(sigmoidf_(gv.y), av.y, v.y);
  v.z = fmaf(sigmoidf_(gv.z), av.z, v.z); v.w = fmaf(sigmoidf_(gv.w), av.w, v.w);
}

template <typename T, int NI>
__global__ void __launch_bounds__(256) gated_add_norm_vec_kernel(GatedNormArgs p) {
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const int W = p.W;
  float* x = p.x + t * W;
  const T* a = p.a ? static_cast<const T*>(p.a) + t * p.lda : nullptr;
  const T* ga = p.ga ? static_cast<const T*>(p.ga) + t * p.ldga : nullptr;
  const T* b = p.b ? static_cast<const T*>(p.b) + t * p.ldb : nullptr;
  const T* gb = p.gb ? static_cast<const T*>(p.gb) + t * p.ldgb : nullptr;
  float4 v[NI];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < W) {
      v[i] = *reinterpret_cast<const float4*>(x + c);
      gated_add4<T>(v[i], a, ga, static_cast<const T*>(p.bias_a), c);
      gated_add4<T>(v[i], b, gb, static_cast<const T*>(p.bias_b), c);
      if (a != nullptr || b != nullptr) *reinterpret_cast<float4*>(x + c) = v[i];
      s += v[i].x + v[i].y + v[i].z + v[i].w;
    }
  }
  const float mean = p.center ? block_sum(s, red) / W : 0.f;
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    if ((threadIdx.x + i * blockDim.x) * 4 < W) {
      v[i].x -= mean; v[i].y -= mean; v[i].z -= mean; v[i].w -= mean;
      q += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
  }
  const float r = rsqrtf(block_sum(q, red) / W + p.eps);
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c < W) {
      const float4 n = make_float4(v[i].x * r, v[i].y * r, v[i].z * r, v[i].w * r);
      float4 w = ld4(static_cast<const T*>(p.w1) + c);
      st4(static_cast<T*>(p.h1) + t * W + c, make_float4(n.x * w.x, n.y * w.y, n.z * w.z, n.w * w.w));
      if (p.h2 != nullptr) {
        w = ld4(static_cast<const T*>(p.w2) + c);
        st4(static_cast<T*>(p.h2) + t * W + c, make_float4(n.x * w.x, n.y * w.y, n.z * w.z, n.w * w.w));
      }
    }
  }
}

template <typename T>
__device__ __forceinline__ float gated_term(const T* a, const T* g, const T* bias, int c) {
  if (a == nullptr) return 0.f;
  const float av = ld(a + c);
  if (g == nullptr) return av;
  return sigmoidf_(ld(g + c) + (bias != nullptr ? ld(bias + c) : 0.f)) * av;
}

template <typename T>
__global__ void __launch_bounds__(256) gated_add_norm_kernel(GatedNormArgs p) {
  extern __shared__ float row[];                           // [W] + [32]
  const int64_t t = blockIdx.x;
  const int W = p.W;
  float* red = row + W;
  float* x = p.x + t * W;
  const T* a = p.a ? static_cast<const T*>(p.a) + t * p.lda : nullptr;
  const T* ga = p.ga ? static_cast<const T*>(p.ga) + t * p.ldga : nullptr;
  const T* b = p.b ? static_cast<const T*>(p.b) + t * p.ldb : nullptr;
  const T* gb = p.gb ? static_cast<const T*>(p.gb) + t * p.ldgb : nullptr;
  float s = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    const float v = x[c] + gated_term<T>(a, ga, static_cast<const T*>(p.bias_a), c) + gated_term<T>(b, gb, static_cast<const T*>(p.bias_b), c);
    if (a != nullptr || b != nullptr) x[c] = v;
    row[c] = v;
    s += v;
  }
  const float mean = p.center ? block_sum(s, red) / W : 0.f;
  float q = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) { const float v = row[c] - mean; q += v * v; }
  const float r = rsqrtf(block_sum(q, red) / W + p.eps);
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    const float n = (row[c] - mean) * r;
    st(static_cast<T*>(p.h1) + t * W + c, n * ld(static_cast<const T*>(p.w1) + c));
    if (p.h2 != nullptr) st(static_cast<T*>(p.h2) + t * W + c, n * ld(static_cast<const T*>(p.w2) + c));
  }
}

// ---------------------------------------------------------------------------------------------------------------------
// Heads of up to three operands of a token: rotation, then division by the root mean square, then the weight; to a dense output
// (padded with zeros) and / or to the token's slot of a cache.  One CTA per token: the sines and cosines of every operand are
// computed once, then a warp takes one head after the other.
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kRotWarps = 4;

template <typename T>
__global__ void __launch_bounds__(kRotWarps * 32) head_rotary_kernel(HeadRotaryArgs p) {
  extern __shared__ float smem[];                          // [warps][max_d], then (cos, sin) of every part's pairs
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t t = blockIdx.x;
  const int pos = static_cast<int>(p.positions[t]);
  float* buf = smem + warp * p.max_d;
  float* tab = smem + kRotWarps * p.max_d;
  int at = 0;
  for (int k = 0; k < p.n_parts; ++k) {
    const RotPart& r = p.part[k];
    if (r.shares_table) continue;
    for (int i = threadIdx.x; i < r.n_turn; i += blockDim.x) {
      float sn, cs;
      turn_angle(r.turns + 2 * i, pos, &sn, &cs);
      cs *= r.amplitude;
      sn *= r.back ? -r.amplitude : r.amplitude;
      tab[2 * (at + i)] = cs;
      tab[2 * (at + i) + 1] = sn;
      if (r.table != nullptr) *reinterpret_cast<float2*>(r.table + 2 * (t * r.n_turn + i)) = make_float2(cs, sn);
    }
    at += r.n_turn;
  }
  __syncthreads();
  int64_t slot = 0;
  if (p.slots != nullptr) slot = p.slots[t];
  int first = 0, tab0 = 0, tab_next = 0;
  for (int k = 0; k < p.n_parts; ++k) {
    const RotPart& r = p.part[k];
    if (!r.shares_table) { tab0 = tab_next; tab_next += r.n_turn; }
    const float* cs = tab + 2 * tab0;
    const int n = r.n_turn;
    const float inv_d = 1.f / static_cast<float>(r.d);
    for (int h = (warp + kRotWarps - first % kRotWarps) % kRotWarps; h < r.heads; h += kRotWarps) {
      const T* x = static_cast<const T*>(r.x) + t * r.ld_x + h * r.hs_x;
      for (int c = lane; c < r.d; c += 32) buf[c] = ld(x + c);
      __syncwarp();
      for (int i = lane; i < n; i += 32) {
        const int a = r.interleaved ? 2 * i : i, b = r.interleaved ? 2 * i + 1 : i + n;
        const float u = buf[a], w = buf[b], c = cs[2 * i], s = cs[2 * i + 1];
        buf[a] = u * c - w * s;
        buf[b] = w * c + u * s;
      }
      __syncwarp();
      float f = 1.f;
      if (r.rms) {
        float ss = 0.f;
        for (int c = lane; c < r.d; c += 32) ss = fmaf(buf[c], buf[c], ss);
        f = rsqrtf(warp_sum(ss) * inv_d + p.eps);
      }
      T* out = r.out != nullptr ? static_cast<T*>(r.out) + t * r.ld_out + h * r.hs_out : nullptr;
      T* page = r.pages != nullptr ? static_cast<T*>(r.pages) + slot * r.ld_page + h * r.hs_page : nullptr;
      for (int c = lane; c < r.d; c += 32) {
        float v = buf[c] * f;
        if (r.weight != nullptr) v *= ld(static_cast<const T*>(r.weight) + c);
        if (out != nullptr) st(out + (r.out_half > 0 && 2 * c >= r.d ? r.out_half + c - r.d / 2 : c), v);
        if (page != nullptr) st(page + c, v);
      }
      if (out != nullptr) {
        if (r.out_half > 0) {
          for (int c = r.d / 2 + lane; c < r.out_half; c += 32) st(out + c, 0.f);
          for (int c = r.out_half + r.d - r.d / 2 + lane; c < r.d_out; c += 32) st(out + c, 0.f);
        } else {
          for (int c = r.d + lane; c < r.d_out; c += 32) st(out + c, 0.f);
        }
      }
      __syncwarp();
    }
    first += r.heads;
  }
}

// ---------------------------------------------------------------------------------------------------------------------
// q_out = [q_n | R q_r | 0], k_out = [k | k_rot | 0] (k_rot common to the heads), v_out = [v | 0]; one CTA per token.
// ---------------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) latent_head_assemble_kernel(LatentHeadArgs p) {
  extern __shared__ float tab[];                           // (cos, sin) of the pairs
  const int64_t t = blockIdx.x;
  const int pos = static_cast<int>(p.positions[t]);
  for (int i = threadIdx.x; i < p.n_turn; i += blockDim.x) {
    float sn, cs;
    turn_angle(p.turns + 2 * i, pos, &sn, &cs);
    tab[2 * i] = cs * p.amplitude;
    tab[2 * i + 1] = sn * p.amplitude;
  }
  __syncthreads();
  const int d = p.d, n = p.n, W = p.width, np = p.n_turn;
  const T* q = static_cast<const T*>(p.q) + t * p.ld_q;
  const T* k = static_cast<const T*>(p.k) + t * p.H * d;
  const T* v = static_cast<const T*>(p.v) + t * p.H * p.dv;
  const T* kr = static_cast<const T*>(p.k_rot) + t * p.ld_kr;
  T* qo = static_cast<T*>(p.q_out) + t * p.H * W;
  T* ko = static_cast<T*>(p.k_out) + t * p.H * W;
  T* vo = static_cast<T*>(p.v_out) + t * p.H * W;
  for (int i = threadIdx.x; i < p.H * W; i += blockDim.x) {
    const int h = i / W, c = i % W, e = c - d;
    float qv = 0.f, kv = 0.f;
    if (e < 0) {
      qv = ld(q + h * (d + n) + c);
      kv = ld(k + h * d + c);
    } else if (e < n) {
      const T* qr = q + h * (d + n) + d;
      kv = ld(kr + e);
      if (e >= 2 * np) {
        qv = ld(qr + e);
      } else {
        const int pr = p.interleaved ? e >> 1 : (e < np ? e : e - np);
        const bool second = p.interleaved ? (e & 1) : e >= np;
        const int a = p.interleaved ? 2 * pr : pr, b = p.interleaved ? 2 * pr + 1 : pr + np;
        const float u = ld(qr + a), w = ld(qr + b), cs = tab[2 * pr], sn = tab[2 * pr + 1];
        qv = second ? w * cs + u * sn : u * cs - w * sn;
      }
    }
    st(qo + i, qv);
    st(ko + i, kv);
    st(vo + i, c < p.dv ? ld(v + h * p.dv + c) : 0.f);
  }
}

template <typename TI, typename T>
__global__ void __launch_bounds__(256) head_gate_kernel(const TI* __restrict__ o, int64_t ldo, int64_t hso, const T* __restrict__ gate,
                                                        int64_t ldg, int elementwise, T* __restrict__ y, int64_t total, int H, int dv) {
  const int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const int64_t th = i / dv, t = th / H;
  const int c = static_cast<int>(i - th * dv), h = static_cast<int>(th - t * H);
  st(y + i, ld(o + t * ldo + h * hso + c) * sigmoidf_(ld(gate + t * ldg + (elementwise ? h * dv + c : h))));
}

// four columns per thread (dv a multiple of 4, aligned rows)
template <typename TI, typename T>
__global__ void __launch_bounds__(256) head_gate_vec_kernel(const TI* __restrict__ o, int64_t ldo, int64_t hso, const T* __restrict__ gate,
                                                            int64_t ldg, int elementwise, T* __restrict__ y, int64_t total4, int H, int dv4) {
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < total4; i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t th = i / dv4;
    const int t = static_cast<int>(th / H), h = static_cast<int>(th - static_cast<int64_t>(t) * H), c = static_cast<int>(i - th * dv4) * 4;
    const float4 v = ld4(o + t * ldo + h * hso + c);
    float4 g;
    if (elementwise) {
      g = ld4(gate + t * ldg + h * dv4 * 4 + c);
      g = make_float4(sigmoidf_(g.x), sigmoidf_(g.y), sigmoidf_(g.z), sigmoidf_(g.w));
    } else {
      const float f = sigmoidf_(ld(gate + t * ldg + h));
      g = make_float4(f, f, f, f);
    }
    st4(y + i * 4, make_float4(v.x * g.x, v.y * g.y, v.z * g.z, v.w * g.w));
  }
}

}  // namespace

bool gated_add_norm(const GatedNormArgs& p, int n_tok, bool bf16, cudaStream_t s) {
  if (n_tok == 0) return true;
  const int W = p.W;
  auto ok = [&](const void* ptr, int64_t ld) {             // four columns at a time
    return ptr == nullptr || (ld % 4 == 0 && reinterpret_cast<uintptr_t>(ptr) % 16 == 0);
  };
  if (W % 4 == 0 && W <= 8192 && ok(p.x, W) && ok(p.a, p.lda) && ok(p.ga, p.ldga) && ok(p.b, p.ldb) && ok(p.gb, p.ldgb) && ok(p.bias_a, 0) &&
      ok(p.bias_b, 0) && ok(p.w1, 0) && ok(p.w2, 0) && ok(p.h1, W) && ok(p.h2, W)) {
    const int threads = std::min(256, (W / 4 + 31) / 32 * 32);
    const int ni = (W / 4 + threads - 1) / threads;
    SEQ_DISPATCH_T(bf16, {
      if (ni <= 1) gated_add_norm_vec_kernel<T, 1><<<n_tok, threads, 0, s>>>(p);
      else if (ni <= 2) gated_add_norm_vec_kernel<T, 2><<<n_tok, threads, 0, s>>>(p);
      else if (ni <= 4) gated_add_norm_vec_kernel<T, 4><<<n_tok, threads, 0, s>>>(p);
      else gated_add_norm_vec_kernel<T, 8><<<n_tok, threads, 0, s>>>(p);
    });
    return true;
  }
  const size_t smem = (static_cast<size_t>(W) + 32) * sizeof(float);
  if (smem > 48 * 1024) return false;
  SEQ_DISPATCH_T(bf16, gated_add_norm_kernel<T><<<n_tok, 256, smem, s>>>(p));
  return true;
}

bool head_rotary(HeadRotaryArgs p, int n_tok, bool bf16, cudaStream_t s) {
  if (n_tok == 0) return true;
  int pairs = 0;
  p.max_d = 1;
  for (int k = 0; k < p.n_parts; ++k) {
    RotPart& r = p.part[k];
    p.max_d = std::max(p.max_d, r.d);
    const RotPart* prev = k > 0 ? &p.part[k - 1] : nullptr;
    r.shares_table = prev != nullptr && prev->n_turn == r.n_turn && prev->turns == r.turns && prev->amplitude == r.amplitude && prev->back == r.back &&
                      r.table == nullptr;
    if (!r.shares_table) pairs += r.n_turn;
  }
  const size_t smem = (static_cast<size_t>(kRotWarps) * p.max_d + 2 * static_cast<size_t>(pairs)) * sizeof(float);
  if (smem > 48 * 1024) return false;
  SEQ_DISPATCH_T(bf16, head_rotary_kernel<T><<<n_tok, kRotWarps * 32, smem, s>>>(p));
  return true;
}

bool latent_head_assemble(const LatentHeadArgs& p, int n_tok, bool bf16, cudaStream_t s) {
  if (n_tok == 0) return true;
  const size_t smem = 2 * static_cast<size_t>(p.n_turn) * sizeof(float);
  if (smem > 48 * 1024) return false;
  SEQ_DISPATCH_T(bf16, latent_head_assemble_kernel<T><<<n_tok, 256, smem, s>>>(p));
  return true;
}

template <typename TI, typename T>
static void launch_head_gate(const void* o, int64_t ldo, int64_t hso, const void* gate, int64_t ldg, bool elementwise, void* y, int64_t total, int H,
                             int dv, cudaStream_t s) {
  const TI* op = static_cast<const TI*>(o);
  const T* gp = static_cast<const T*>(gate);
  T* yp = static_cast<T*>(y);
  const bool gate_ok = !elementwise || (ldg % 4 == 0 && reinterpret_cast<uintptr_t>(gate) % (4 * sizeof(T)) == 0);
  if (dv % 4 == 0 && ldo % 4 == 0 && hso % 4 == 0 && reinterpret_cast<uintptr_t>(o) % 16 == 0 && reinterpret_cast<uintptr_t>(y) % 16 == 0 && gate_ok) {
    const unsigned blocks = static_cast<unsigned>(std::min<int64_t>((total / 4 + 255) / 256, 148 * 32));
    head_gate_vec_kernel<TI, T><<<blocks, 256, 0, s>>>(op, ldo, hso, gp, ldg, elementwise, yp, total / 4, H, dv / 4);
  } else {
    head_gate_kernel<TI, T><<<static_cast<unsigned>((total + 255) / 256), 256, 0, s>>>(op, ldo, hso, gp, ldg, elementwise, yp, total, H, dv);
  }
}

void head_gate(const void* o, bool o_f32, int64_t ldo, int64_t hso, const void* gate, int64_t ldg, bool elementwise, void* y, int n_tok, int H,
               int dv, bool bf16, cudaStream_t s) {
  const int64_t total = static_cast<int64_t>(n_tok) * H * dv;
  if (total == 0) return;
  SEQ_DISPATCH_T(bf16, {
    if (o_f32) launch_head_gate<float, T>(o, ldo, hso, gate, ldg, elementwise, y, total, H, dv, s);
    else launch_head_gate<T, T>(o, ldo, hso, gate, ldg, elementwise, y, total, H, dv, s);
  });
}

}  // namespace b200seq
