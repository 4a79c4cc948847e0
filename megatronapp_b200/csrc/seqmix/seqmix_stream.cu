// Kernels of layers over several fp32 residual streams with a sliding-window attention beside a selective scan (sm_100a):
// the stream update fused with the layer norm of the next sublayer's input, sinusoidal positions added to an fp32 embedding, an
// RMS norm per head, paged grouped-query attention with a distance penalty per head, a sliding window, an optional sink in the
// softmax denominator and a scalar output gate per head, and the selective scan (one decay per channel and state).
//
// Conventions as in seqmix.cu: activations are `T` (float or __nv_bfloat16); statistics, angles, scores, weights, gates, decays,
// step sizes and every recurrent state are fp32; `cu[R + 1]` / `rows[R]` describe the packed batch.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>
#include <algorithm>

#include "seq_common.cuh"
#include "seq_window.cuh"
#include "seqmix_api.h"

namespace b200seq {

namespace {

using namespace dev;

__device__ __forceinline__ float block_sum(float v, float* red) {   // every thread gets the sum; red holds >= 32 floats
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < (blockDim.x >> 5); ++i) tot += red[i];
  return tot;
}

// ---------------------------------------------------------------------------------------------------------------------
// Streams X [T, S, W] (fp32, in place).  With a pending sublayer output: y = ls * (sa * (a + bias_a) + sb * b) and
// X_t <- sum_s mix[s, t] X_s + out[t] * y for all t at once.  Then, with `inp`: u = sum_s inp[s] X_s and
// h = (u - mean) / sqrt(var + eps) * w + beta (or u / sqrt(mean(u^2) + eps) * w without beta).  One CTA per token.
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kMaxStreams = 16;

template <typename T>
__global__ void __launch_bounds__(256) stream_mix_norm_kernel(StreamNormArgs p) {
  extern __shared__ float su[];                      // [W]
  __shared__ float red[32];
  __shared__ float cmix[kMaxStreams * kMaxStreams], cout_[kMaxStreams], cin[kMaxStreams];
  const int S = p.S, W = p.W;
  if (threadIdx.x < S * S && p.mix != nullptr) cmix[threadIdx.x] = p.mix[threadIdx.x];
  if (threadIdx.x < S) {
    if (p.outc != nullptr) cout_[threadIdx.x] = p.outc[threadIdx.x];
    if (p.inp != nullptr) cin[threadIdx.x] = p.inp[threadIdx.x];
  }
  __syncthreads();
  const int64_t row = blockIdx.x;
  float* X = p.x + row * S * W;
  const T* a = static_cast<const T*>(p.a);
  const T* b = static_cast<const T*>(p.b);
  const T* ba = static_cast<const T*>(p.bias_a);
  const T* ls = static_cast<const T*>(p.ls);
  float sum = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    float xs[kMaxStreams];
#pragma unroll
    for (int s = 0; s < kMaxStreams; ++s) xs[s] = s < S ? X[static_cast<int64_t>(s) * W + c] : 0.f;
    if (a != nullptr) {
      float y = ld(a + row * p.lda + c);
      if (ba != nullptr) y += ld(ba + c);
      y *= p.scale_a;
      if (b != nullptr) y = fmaf(p.scale_b, ld(b + row * p.ldb + c), y);
      if (ls != nullptr) y *= ld(ls + c);
      float nx[kMaxStreams];
#pragma unroll
      for (int t = 0; t < kMaxStreams; ++t) {
        if (t < S) {
          float v = cout_[t] * y;
#pragma unroll
          for (int s = 0; s < kMaxStreams; ++s)
            if (s < S) v = fmaf(cmix[s * S + t], xs[s], v);
          nx[t] = v;
        }
      }
#pragma unroll
      for (int t = 0; t < kMaxStreams; ++t)
        if (t < S) { xs[t] = nx[t]; X[static_cast<int64_t>(t) * W + c] = nx[t]; }
    }
    if (p.inp != nullptr) {
      float u = 0.f;
#pragma unroll
      for (int s = 0; s < kMaxStreams; ++s)
        if (s < S) u = fmaf(cin[s], xs[s], u);
      su[c] = u;
      sum += u;
    }
  }
  if (p.inp == nullptr) return;
  const T* w = static_cast<const T*>(p.w);
  const T* beta = static_cast<const T*>(p.beta);
  T* h = static_cast<T*>(p.h) + row * W;
  float mean = 0.f;
  if (beta != nullptr || p.center) mean = block_sum(sum, red) / static_cast<float>(W);
  else __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) { const float d = su[c] - mean; ss = fmaf(d, d, ss); }
  const float rstd = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(W) + p.eps);
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    float v = (su[c] - mean) * rstd * ld(w + c);
    if (beta != nullptr) v += ld(beta + c);
    st(h + c, v);
  }
}

// Four columns per thread and the number of streams known at compile time (W a multiple of 4, rows 16-byte aligned).
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
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = raw;
}
__device__ __forceinline__ float4 f4_fma(float a, float4 x, float4 y) {
  return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w));
}
__device__ __forceinline__ float4 f4_mul(float4 x, float4 y) { return make_float4(x.x * y.x, x.y * y.y, x.z * y.z, x.w * y.w); }

template <typename T, int S>
__global__ void __launch_bounds__(256) stream_mix_norm_vec_kernel(StreamNormArgs p) {
  extern __shared__ __align__(16) float su[];        // [W]
  __shared__ float red[32];
  const int W = p.W;
  const int64_t row = blockIdx.x;
  float* X = p.x + row * S * W;
  const T* a = static_cast<const T*>(p.a);
  const T* b = static_cast<const T*>(p.b);
  const T* ba = static_cast<const T*>(p.bias_a);
  const T* ls = static_cast<const T*>(p.ls);
  float cmix[S * S], cout_[S], cin[S];
#pragma unroll
  for (int i = 0; i < S * S; ++i) cmix[i] = a != nullptr ? p.mix[i] : 0.f;
#pragma unroll
  for (int i = 0; i < S; ++i) { cout_[i] = a != nullptr ? p.outc[i] : 0.f; cin[i] = p.inp != nullptr ? p.inp[i] : 0.f; }
  float sum = 0.f;
  for (int c = threadIdx.x * 4; c < W; c += blockDim.x * 4) {
    float4 xs[S];
#pragma unroll
    for (int s = 0; s < S; ++s) xs[s] = *reinterpret_cast<const float4*>(X + static_cast<int64_t>(s) * W + c);
    if (a != nullptr) {
      float4 y = ld4(a + row * p.lda + c);
      if (ba != nullptr) { const float4 bv = ld4(ba + c); y = make_float4(y.x + bv.x, y.y + bv.y, y.z + bv.z, y.w + bv.w); }
      y = make_float4(y.x * p.scale_a, y.y * p.scale_a, y.z * p.scale_a, y.w * p.scale_a);
      if (b != nullptr) y = f4_fma(p.scale_b, ld4(b + row * p.ldb + c), y);
      if (ls != nullptr) y = f4_mul(y, ld4(ls + c));
      float4 nx[S];
#pragma unroll
      for (int t = 0; t < S; ++t) {
        float4 v = make_float4(cout_[t] * y.x, cout_[t] * y.y, cout_[t] * y.z, cout_[t] * y.w);
#pragma unroll
        for (int s = 0; s < S; ++s) v = f4_fma(cmix[s * S + t], xs[s], v);
        nx[t] = v;
      }
#pragma unroll
      for (int t = 0; t < S; ++t) { xs[t] = nx[t]; *reinterpret_cast<float4*>(X + static_cast<int64_t>(t) * W + c) = nx[t]; }
    }
    if (p.inp != nullptr) {
      float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < S; ++s) u = f4_fma(cin[s], xs[s], u);
      *reinterpret_cast<float4*>(su + c) = u;
      sum += (u.x + u.y) + (u.z + u.w);
    }
  }
  if (p.inp == nullptr) return;
  const T* w = static_cast<const T*>(p.w);
  const T* beta = static_cast<const T*>(p.beta);
  T* h = static_cast<T*>(p.h) + row * W;
  float mean = 0.f;
  if (beta != nullptr || p.center) mean = block_sum(sum, red) / static_cast<float>(W);
  else __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x * 4; c < W; c += blockDim.x * 4) {
    const float4 u = *reinterpret_cast<const float4*>(su + c);
    const float d0 = u.x - mean, d1 = u.y - mean, d2 = u.z - mean, d3 = u.w - mean;
    ss += (d0 * d0 + d1 * d1) + (d2 * d2 + d3 * d3);
  }
  const float rstd = 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(W) + p.eps);
  for (int c = threadIdx.x * 4; c < W; c += blockDim.x * 4) {
    const float4 u = *reinterpret_cast<const float4*>(su + c);
    const float4 wv = ld4(w + c);
    float4 v = make_float4((u.x - mean) * rstd * wv.x, (u.y - mean) * rstd * wv.y, (u.z - mean) * rstd * wv.z, (u.w - mean) * rstd * wv.w);
    if (beta != nullptr) { const float4 bv = ld4(beta + c); v = make_float4(v.x + bv.x, v.y + bv.y, v.z + bv.z, v.w + bv.w); }
    st4(h + c, v);
  }
}

// x [T, W] (fp32, in place): x[t, 2i] += sin(pos_t * f_i), x[t, 2i + 1] += cos(pos_t * f_i)
__global__ void add_sinusoid_kernel(float* __restrict__ x, const int64_t* __restrict__ positions, const float* __restrict__ freq,
                                    int64_t n_pairs_total, int half) {
  const int64_t idx = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (idx >= n_pairs_total) return;
  const int64_t t = idx / half;
  const int i = static_cast<int>(idx % half);
  const float ang = static_cast<float>(positions[t]) * freq[i];
  float sn, cs;
  sincosf(ang, &sn, &cs);
  float2* px = reinterpret_cast<float2*>(x + t * (2 * static_cast<int64_t>(half))) + i;
  float2 v = *px;
  v.x += sn; v.y += cs;
  *px = v;
}

// x [T, heads, d] (row stride ldx) -> y contiguous: every head divided by its root mean square over d, times w [d]
template <typename T>
__global__ void __launch_bounds__(128) head_rms_norm_kernel(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w,
                                                            T* __restrict__ y, int64_t rows, int heads, int d, float eps) {
  const int64_t row = static_cast<int64_t>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  if (row >= rows) return;
  const int lane = threadIdx.x & 31;
  const int64_t t = row / heads;
  const int h = static_cast<int>(row % heads);
  const T* src = x + t * ldx + static_cast<int64_t>(h) * d;
  float ss = 0.f;
  for (int c = lane; c < d; c += 32) { const float v = ld(src + c); ss = fmaf(v, v, ss); }
  ss = warp_sum(ss);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(d) + eps);
  for (int c = lane; c < d; c += 32) st(y + row * d + c, ld(src + c) * r * ld(w + c));
}

// ---------------------------------------------------------------------------------------------------------------------
// Selective scan.  Per channel c and state n:  S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;  y_c = sum_n S[c, n] C_n +
// D_c x_c, then y * silu(z) * out_scale.  dt = softplus(dt_pre + dt_bias), A = -exp(A_log).
// grid (channel blocks of 32, sequences).  The N states of a channel are spread over 4 adjacent lanes (state n on lane n % 4);
// dt, x, B and C of 16 tokens are staged in shared memory per round, so the sequential part touches registers and shared
// memory only.
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kSelThreads = 128, kSelParts = 4, kSelCh = kSelThreads / kSelParts, kSelChunk = 16;

template <typename T, int NS>
__global__ void __launch_bounds__(kSelThreads) selective_scan_kernel(SelScanArgs p) {
  extern __shared__ float smem[];
  const int N = p.N;
  float* sdt = smem;                                 // [chunk][32]
  float* sx = sdt + kSelChunk * kSelCh;              // [chunk][32]
  float* sz = sx + kSelChunk * kSelCh;               // [chunk][32]  silu(z) * out_scale
  float* sy = sz + kSelChunk * kSelCh;               // [chunk][32]  outputs of the round
  float* sB = sy + kSelChunk * kSelCh;               // [chunk][N]
  float* sC = sB + kSelChunk * N;                    // [chunk][N]
  const int r = blockIdx.y, part = threadIdx.x & (kSelParts - 1), cl = threadIdx.x >> 2;
  const int c0 = blockIdx.x * kSelCh, c = c0 + cl;
  const bool live = c < p.C;
  const int a = p.cu[r], b = p.cu[r + 1];
  if (a >= b) return;
  const T* x = static_cast<const T*>(p.x);
  const T* z = static_cast<const T*>(p.z);
  const T* Bm = static_cast<const T*>(p.B);
  const T* Cm = static_cast<const T*>(p.Cm);
  T* y = static_cast<T*>(p.y);
  float A[NS], S[NS];
  float* st_row = p.state + (static_cast<int64_t>(p.rows[r]) * p.C + (live ? c : 0)) * N;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = part + kSelParts * i;
    const bool ok = live && n < N;
    // decay exp(dt * A) = 2^(dt * A * log2 e), A = -exp(A_log)
    A[i] = ok ? -expf(ld(static_cast<const T*>(p.A_log) + static_cast<int64_t>(c) * N + n)) * 1.4426950408889634f : 0.f;
    S[i] = ok ? st_row[n] : 0.f;
  }
  const float Dc = live ? ld(static_cast<const T*>(p.D) + c) : 0.f;
  for (int t0 = a; t0 < b; t0 += kSelChunk) {
    const int nt = min(kSelChunk, b - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * kSelCh; i += kSelThreads) {
      const int tt = i / kSelCh, cc = i % kSelCh;
      float dtv = 0.f, xv = 0.f, zg = p.out_scale;
      if (c0 + cc < p.C) {
        if (z != nullptr) { const float zv = ld(z + static_cast<int64_t>(t0 + tt) * p.ldz + c0 + cc); zg *= zv * sigmoidf_(zv); }
        const float pre = p.dt_pre[static_cast<int64_t>(t0 + tt) * p.lddt + c0 + cc] +
                          (p.dt_bias != nullptr ? ld(static_cast<const T*>(p.dt_bias) + c0 + cc) : 0.f);
        dtv = pre > 20.f ? pre : log1pf(expf(pre));
        xv = ld(x + static_cast<int64_t>(t0 + tt) * p.ldx + c0 + cc);
      }
      sdt[i] = dtv; sx[i] = xv; sz[i] = zg;
    }
    for (int i = threadIdx.x; i < nt * N; i += kSelThreads) {
      const int tt = i / N, n = i % N;
      sB[i] = ld(Bm + static_cast<int64_t>(t0 + tt) * p.ldb + n);
      sC[i] = ld(Cm + static_cast<int64_t>(t0 + tt) * p.ldc + n);
    }
    __syncthreads();
    for (int tt = 0; tt < nt; ++tt) {
      const float dtv = sdt[tt * kSelCh + cl], xv = sx[tt * kSelCh + cl];
      const float dx = dtv * xv;
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        const int n = part + kSelParts * i;
        if (n < N) {
          S[i] = fmaf(exp2f(dtv * A[i]), S[i], dx * sB[tt * N + n]);
          acc = fmaf(S[i], sC[tt * N + n], acc);
        }
      }
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      if (part == 0) sy[tt * kSelCh + cl] = fmaf(Dc, xv, acc) * sz[tt * kSelCh + cl];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * kSelCh; i += kSelThreads) {
      const int tt = i / kSelCh, cc = i % kSelCh;
      if (c0 + cc < p.C) st(y + static_cast<int64_t>(t0 + tt) * p.ldy + c0 + cc, sy[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = part + kSelParts * i;
    if (live && n < N) st_row[n] = S[i];
  }
}

}  // namespace

// ---------------------------------------------------------------------------------------------------------------------
// launchers
// ---------------------------------------------------------------------------------------------------------------------
bool stream_mix_norm(const StreamNormArgs& p, int n_tok, bool bf16, cudaStream_t s) {
  if (p.S < 1 || p.S > kMaxStreams) return false;
  if (n_tok == 0) return true;
  const size_t smem = p.inp != nullptr ? static_cast<size_t>(p.W) * sizeof(float) : 0;
  if (smem > 200 * 1024) return false;
  const size_t esz = bf16 ? 2 : 4;
  auto al = [&](const void* q, size_t bytes) { return q == nullptr || reinterpret_cast<uintptr_t>(q) % bytes == 0; };
  const bool vec = p.W % 4 == 0 && p.S <= 4 && al(p.x, 16) && al(p.a, 4 * esz) && al(p.b, 4 * esz) && al(p.bias_a, 4 * esz) &&
                   al(p.ls, 4 * esz) && al(p.w, 4 * esz) && al(p.beta, 4 * esz) && al(p.h, 4 * esz) && p.lda % 4 == 0 && p.ldb % 4 == 0;
#define SEQ_STREAM_VEC(SS)                                                                                                  \
  {                                                                                                                         \
    if (smem > 48 * 1024)                                                                                                   \
      cudaFuncSetAttribute(stream_mix_norm_vec_kernel<T, SS>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)); \
    stream_mix_norm_vec_kernel<T, SS><<<n_tok, 256, smem, s>>>(p);                                                          \
  }
  SEQ_DISPATCH_T(bf16, {
    if (vec && p.S == 1) SEQ_STREAM_VEC(1)
    else if (vec && p.S == 2) SEQ_STREAM_VEC(2)
    else if (vec && p.S == 3) SEQ_STREAM_VEC(3)
    else if (vec && p.S == 4) SEQ_STREAM_VEC(4)
    else {
      if (smem > 48 * 1024)
        cudaFuncSetAttribute(stream_mix_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
      stream_mix_norm_kernel<T><<<n_tok, 256, smem, s>>>(p);
    }
  });
#undef SEQ_STREAM_VEC
  return true;
}

void add_sinusoid(float* x, const int64_t* positions, const float* freq, int n_tok, int width, cudaStream_t s) {
  const int half = width / 2;
  const int64_t n = static_cast<int64_t>(n_tok) * half;
  if (n == 0) return;
  add_sinusoid_kernel<<<static_cast<unsigned>((n + 255) / 256), 256, 0, s>>>(x, positions, freq, n, half);
}

void head_rms_norm(const void* x, int64_t ldx, const void* w, void* y, int n_tok, int heads, int d, float eps, bool bf16,
                   cudaStream_t s) {
  const int64_t rows = static_cast<int64_t>(n_tok) * heads;
  if (rows == 0) return;
  SEQ_DISPATCH_T(bf16, head_rms_norm_kernel<T><<<static_cast<unsigned>((rows + 3) / 4), 128, 0, s>>>(
                           static_cast<const T*>(x), ldx, static_cast<const T*>(w), static_cast<T*>(y), rows, heads, d, eps));
}


int window_attention_splits(int H, int G, int n_tok, int max_keys) {
  const int rep = H / G, hc = std::min(rep, kDecMaxHeads);
  const int ctas = n_tok * G * ((rep + hc - 1) / hc);
  const int by_keys = (max_keys + 2 * kWinTile - 1) / (2 * kWinTile);     // at least two tiles per split
  const int by_fill = (8 * 148 + ctas - 1) / ctas;
  return std::max(1, std::min(std::min(by_keys, by_fill), 64));
}

bool window_attention_paged(const WindowAttnArgs& p, bool bf16, cudaStream_t s) { return run_window_attention<false>(p, bf16, s); }

template <typename T, int NS>
static void launch_sel(const SelScanArgs& p, int R, cudaStream_t s) {
  const size_t smem = (4 * static_cast<size_t>(kSelChunk) * kSelCh + 2 * static_cast<size_t>(kSelChunk) * p.N) * sizeof(float);
  dim3 grid((p.C + kSelCh - 1) / kSelCh, R);
  selective_scan_kernel<T, NS><<<grid, kSelThreads, smem, s>>>(p);
}

bool selective_scan(const SelScanArgs& p, int R, bool bf16, cudaStream_t s) {
  if (R == 0) return true;
  if (R > 65535) return false;
  SEQ_DISPATCH_T(bf16, {
    if (p.N <= 16) launch_sel<T, 4>(p, R, s);
    else if (p.N <= 32) launch_sel<T, 8>(p, R, s);
    else if (p.N <= 64) launch_sel<T, 16>(p, R, s);
    else if (p.N <= 128) launch_sel<T, 32>(p, R, s);
    else return false;
  });
  return true;
}

}  // namespace b200seq
