// Real-gated linear recurrent unit with block-diagonal gates (sm_100a), kernels for any size and for fp32:
//   r, i = sigmoid(W_r[b] u_b + b_r), sigmoid(W_i[b] u_b + b_i);  a = exp(-scale * r * softplus(lam))
//   S <- a S + sqrt(1 - a^2) i u;  y = S * gelu_tanh(y_pre)
// The gates' pre-activations are a block-diagonal product with fp32 results in a workspace; the recurrence is linear per channel
// and is cut into runs of kRun tokens: short steps walk a run from the carried state; long ones first reduce every run to (P, Q)
// with S_end = P S_begin + Q, then find each run's S_begin, then walk every run again and write y.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>
#include <algorithm>

#include "seq_common.cuh"
#include "seq_lru.cuh"
#include "seqmix_api.h"

namespace b200seq {

namespace {

using namespace dev;

#define SEQ_DISPATCH_T(is_bf16, ...)                      \
  if (is_bf16) { using T = __nv_bfloat16; __VA_ARGS__; }  \
  else { using T = float; __VA_ARGS__; }

// ---------------------------------------------------------------------------------------------------------------------
// pre[t, g, b * n + o] = sum_k w[b, g, o, k] u[t, b * n + k] + bias[b, g, o].  grid (token tiles, blocks, output tiles); a CTA owns
// 32 tokens x 64 of the 2 n outputs of its block.
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kGateTok = 32, kGateOut = 64, kGateK = 32, kGateThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kGateThreads) lru_gates_kernel(LruArgs p) {
  __shared__ float su[kGateTok][kGateK + 1], sw[kGateOut][kGateK + 1];
  const int n = p.n, b = blockIdx.y, t0 = blockIdx.x * kGateTok, o0 = blockIdx.z * kGateOut;
  const int tx = threadIdx.x % kGateOut, ty = threadIdx.x / kGateOut;           // output, token group of 8
  constexpr int kPer = kGateTok / (kGateThreads / kGateOut);
  float acc[kPer];
#pragma unroll
  for (int j = 0; j < kPer; ++j) acc[j] = 0.f;
  const T* u = static_cast<const T*>(p.u) + b * n;
  const T* w = static_cast<const T*>(p.w) + static_cast<int64_t>(b) * 2 * n * n;
  for (int k0 = 0; k0 < n; k0 += kGateK) {
    __syncthreads();
    for (int i = threadIdx.x; i < kGateTok * kGateK; i += kGateThreads) {
      const int r = i / kGateK, c = i % kGateK;
      su[r][c] = (t0 + r < p.n_tok && k0 + c < n) ? ld(u + static_cast<int64_t>(t0 + r) * p.ldu + k0 + c) : 0.f;
    }
    for (int i = threadIdx.x; i < kGateOut * kGateK; i += kGateThreads) {
      const int r = i / kGateK, c = i % kGateK;
      sw[r][c] = (o0 + r < 2 * n && k0 + c < n) ? ld(w + static_cast<int64_t>(o0 + r) * n + k0 + c) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < kGateK; ++k) {
      const float wv = sw[tx][k];
#pragma unroll
      for (int j = 0; j < kPer; ++j) acc[j] = fmaf(wv, su[ty * kPer + j][k], acc[j]);
    }
  }
  const int o = o0 + tx;
  if (o >= 2 * n) return;
  const float bias = ld(static_cast<const T*>(p.bias) + static_cast<int64_t>(b) * 2 * n + o);
  const int g = o / n, c = b * n + o % n;
#pragma unroll
  for (int j = 0; j < kPer; ++j) {
    const int t = t0 + ty * kPer + j;
    if (t < p.n_tok) p.pre[(static_cast<int64_t>(t) * 2 + g) * p.C + c] = acc[j] + bias;
  }
}

// ---------------------------------------------------------------------------------------------------------------------
// the recurrence; grid (channel blocks, runs, sequences), a thread owns one channel
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kLruThreads = 128, kLruBatch = 8;

template <typename T>
__global__ void __launch_bounds__(kLruThreads) lru_reduce_kernel(LruArgs p) {
  const int c = blockIdx.x * kLruThreads + threadIdx.x, r = blockIdx.z;
  const int a0 = p.cu[r] + blockIdx.y * kLruRun, b0 = min(p.cu[r + 1], a0 + kLruRun);
  if (c >= p.C || a0 >= b0) return;
  const T* up = static_cast<const T*>(p.u);
  const float rate = p.decay_scale * softplusf_(ld(static_cast<const T*>(p.lam) + c));
  float P = 1.f, Q = 0.f;
  for (int64_t t0 = a0; t0 < b0; t0 += kLruBatch) {
    float uv[kLruBatch], rv[kLruBatch], iv[kLruBatch];
#pragma unroll
    for (int j = 0; j < kLruBatch; ++j) {
      const bool in = t0 + j < b0;
      uv[j] = in ? ld(up + (t0 + j) * p.ldu + c) : 0.f;
      rv[j] = in ? p.pre[(t0 + j) * 2 * p.C + c] : 0.f;
      iv[j] = in ? p.pre[((t0 + j) * 2 + 1) * p.C + c] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < kLruBatch; ++j) {
      if (t0 + j < b0) {
        float a, put;
        lru_gates(rv[j], iv[j], uv[j], rate, &a, &put);
        P *= a;
        Q = fmaf(a, Q, put);
      }
    }
  }
  float* ws = p.ws + ((static_cast<int64_t>(r) * p.max_runs + blockIdx.y) * p.C + c) * 2;
  ws[0] = P; ws[1] = Q;
}

__global__ void __launch_bounds__(kLruThreads) lru_carry_kernel(LruArgs p) {
  const int c = blockIdx.x * kLruThreads + threadIdx.x, r = blockIdx.z;
  const int n = p.cu[r + 1] - p.cu[r];
  if (c >= p.C || n <= 0) return;
  float* st_ = p.state + static_cast<int64_t>(p.rows[r]) * p.C + c;
  float S = *st_;
  const int runs = (n + kLruRun - 1) / kLruRun;
  for (int y = 0; y < runs; ++y) {
    float* ws = p.ws + ((static_cast<int64_t>(r) * p.max_runs + y) * p.C + c) * 2;
    const float P = ws[0], Q = ws[1];
    ws[0] = S;                                             // the run's starting state
    S = fmaf(P, S, Q);
  }
  *st_ = S;
}

template <typename T, bool CARRIED>
__global__ void __launch_bounds__(kLruThreads) lru_apply_kernel(LruArgs p) {
  const int c = blockIdx.x * kLruThreads + threadIdx.x, r = blockIdx.z;
  const int lo = p.cu[r], hi = p.cu[r + 1];
  const int a0 = CARRIED ? lo + blockIdx.y * kLruRun : lo, b0 = CARRIED ? min(hi, a0 + kLruRun) : hi;
  if (c >= p.C || a0 >= b0) return;
  const T* up = static_cast<const T*>(p.u);
  const T* yp = static_cast<const T*>(p.y_pre);
  T* y = static_cast<T*>(p.y);
  const float rate = p.decay_scale * softplusf_(ld(static_cast<const T*>(p.lam) + c));
  float* st_ = p.state + static_cast<int64_t>(p.rows[r]) * p.C + c;
  float S = CARRIED ? p.ws[((static_cast<int64_t>(r) * p.max_runs + blockIdx.y) * p.C + c) * 2] : *st_;
  for (int64_t t0 = a0; t0 < b0; t0 += kLruBatch) {
    float uv[kLruBatch], rv[kLruBatch], iv[kLruBatch], yv[kLruBatch];
#pragma unroll
    for (int j = 0; j < kLruBatch; ++j) {
      const bool in = t0 + j < b0;
      uv[j] = in ? ld(up + (t0 + j) * p.ldu + c) : 0.f;
      rv[j] = in ? p.pre[(t0 + j) * 2 * p.C + c] : 0.f;
      iv[j] = in ? p.pre[((t0 + j) * 2 + 1) * p.C + c] : 0.f;
      yv[j] = (in && yp != nullptr) ? ld(yp + (t0 + j) * p.ldy + c) : 0.f;
    }
#pragma unroll
    for (int j = 0; j < kLruBatch; ++j) {
      if (t0 + j < b0) {
        float a, put;
        lru_gates(rv[j], iv[j], uv[j], rate, &a, &put);
        S = fmaf(a, S, put);
        st(y + (t0 + j) * p.C + c, yp != nullptr ? S * gelu_tanhf_(yv[j]) : S);
      }
    }
  }
  if (!CARRIED) *st_ = S;
}

// ---------------------------------------------------------------------------------------------------------------------
// A decoding batch, one token per sequence: grid (blocks, 32-channel slices, groups of 16 sequences).  Lane = output channel, a warp
// carries four sequences; both gates' rows of the slice and the sequences' inputs are staged 128 wide in shared memory, 16-byte loads where rows allow.
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kStepSeq = 16, kStepK = 128, kStepWarps = 4, kStepPer = kStepSeq / kStepWarps;

template <typename T>
__global__ void __launch_bounds__(kStepWarps * 32) lru_step_kernel(LruArgs p, int R) {
  __shared__ float2 sw[kStepK][33];                        // (recurrence, input) weight of [k][channel]
  __shared__ __align__(16) float su[kStepSeq][kStepK];
  __shared__ int tok[kStepSeq];                            // packed token of each sequence, -1: none
  const int n = p.n, b = blockIdx.x, o0 = blockIdx.y * 32, r0 = blockIdx.z * kStepSeq;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* w = static_cast<const T*>(p.w) + static_cast<int64_t>(b) * 2 * n * n;
  const T* u = static_cast<const T*>(p.u) + b * n;
  if (threadIdx.x < kStepSeq) {
    const int r = r0 + threadIdx.x;
    tok[threadIdx.x] = (r < R && p.cu[r] < p.cu[r + 1]) ? p.cu[r] : -1;
  }
  float ar[kStepPer], ai[kStepPer];
#pragma unroll
  for (int j = 0; j < kStepPer; ++j) ar[j] = ai[j] = 0.f;
  // what the epilogue needs is on its way while the gates are summed
  __syncthreads();
  const int o = o0 + lane, c = b * n + min(o, n - 1);
  const bool live = o < n;
  const T* bias = static_cast<const T*>(p.bias) + static_cast<int64_t>(b) * 2 * n + min(o, n - 1);
  const float br = ld(bias), bi = ld(bias + n), rate = p.decay_scale * softplusf_(ld(static_cast<const T*>(p.lam) + c));
  int t_[kStepPer];
  float uv_[kStepPer], y_[kStepPer], s_[kStepPer];
  float* st_[kStepPer];
#pragma unroll
  for (int j = 0; j < kStepPer; ++j) {
    t_[j] = tok[warp * kStepPer + j];
    uv_[j] = y_[j] = s_[j] = 0.f;
    st_[j] = nullptr;
    if (t_[j] >= 0) {
      st_[j] = p.state + static_cast<int64_t>(p.rows[r0 + warp * kStepPer + j]) * p.C + c;
      s_[j] = *st_[j];
      uv_[j] = ld(static_cast<const T*>(p.u) + static_cast<int64_t>(t_[j]) * p.ldu + c);
      if (p.y_pre != nullptr) y_[j] = ld(static_cast<const T*>(p.y_pre) + static_cast<int64_t>(t_[j]) * p.ldy + c);
    }
  }
  for (int k0 = 0; k0 < n; k0 += kStepK) {
    __syncthreads();
    constexpr int V = 16 / sizeof(T);                      // lane = channel: the shared-memory stores of a step are conflict-free
    if (n % V == 0 && reinterpret_cast<uintptr_t>(p.w) % 16 == 0) {
#pragma unroll
      for (int q = 0; q < kStepK / V / kStepWarps; ++q) {
        const int k = (warp + q * kStepWarps) * V, o = o0 + lane;
        union { uint4 raw; T v[V]; } wr, wi;
        wr.raw = wi.raw = make_uint4(0u, 0u, 0u, 0u);
        if (o < n && k0 + k < n) {
          const T* src = w + static_cast<int64_t>(o) * n + k0 + k;
          wr.raw = *reinterpret_cast<const uint4*>(src);
          wi.raw = *reinterpret_cast<const uint4*>(src + static_cast<int64_t>(n) * n);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) sw[k + e][lane] = make_float2(ld(&wr.v[e]), ld(&wi.v[e]));
      }
    } else {
      for (int i = threadIdx.x; i < 32 * kStepK; i += kStepWarps * 32) {
        const int o = i / kStepK, k = i % kStepK;
        const bool in = o0 + o < n && k0 + k < n;
        const int64_t at = static_cast<int64_t>(o0 + o) * n + k0 + k;
        sw[k][o] = in ? make_float2(ld(w + at), ld(w + at + static_cast<int64_t>(n) * n)) : make_float2(0.f, 0.f);
      }
    }
#pragma unroll
    for (int q = 0; q < kStepSeq * kStepK / (kStepWarps * 32); ++q) {
      const int i = threadIdx.x + q * kStepWarps * 32, r = i / kStepK, k = i % kStepK;
      su[r][k] = (tok[r] >= 0 && k0 + k < n) ? ld(u + static_cast<int64_t>(tok[r]) * p.ldu + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll 4
    for (int k = 0; k < kStepK; k += 4) {
      float2 wv[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) wv[e] = sw[k + e][lane];
#pragma unroll
      for (int j = 0; j < kStepPer; ++j) {
        const float4 uv = *reinterpret_cast<const float4*>(&su[warp * kStepPer + j][k]);
        ar[j] = fmaf(wv[0].x, uv.x, ar[j]); ai[j] = fmaf(wv[0].y, uv.x, ai[j]);
        ar[j] = fmaf(wv[1].x, uv.y, ar[j]); ai[j] = fmaf(wv[1].y, uv.y, ai[j]);
        ar[j] = fmaf(wv[2].x, uv.z, ar[j]); ai[j] = fmaf(wv[2].y, uv.z, ai[j]);
        ar[j] = fmaf(wv[3].x, uv.w, ar[j]); ai[j] = fmaf(wv[3].y, uv.w, ai[j]);
      }
    }
  }
#pragma unroll
  for (int j = 0; j < kStepPer; ++j) {
    if (!live || t_[j] < 0) continue;
    float a, put;
    lru_gates(ar[j] + br, ai[j] + bi, uv_[j], rate, &a, &put);
    const float S = fmaf(a, s_[j], put);
    *st_[j] = S;
    st(static_cast<T*>(p.y) + static_cast<int64_t>(t_[j]) * p.C + c, p.y_pre != nullptr ? S * gelu_tanhf_(y_[j]) : S);
  }
}

}  // namespace

bool rglru_step(const LruArgs& p, int R, bool bf16, cudaStream_t s) {
  if (R == 0 || p.n_tok == 0 || p.C == 0) return true;
  const dim3 grid(p.n_blocks, (p.n + 31) / 32, (R + kStepSeq - 1) / kStepSeq);
  if (grid.y > 65535 || grid.z > 65535) return false;
  SEQ_DISPATCH_T(bf16, lru_step_kernel<T><<<grid, kStepWarps * 32, 0, s>>>(p, R));
  return true;
}

int lru_runs(int max_len) { return max_len <= kLruRun ? 1 : (max_len + kLruRun - 1) / kLruRun; }

bool rglru_scan(const LruArgs& p, int R, bool bf16, cudaStream_t s) {
  if (R == 0 || p.n_tok == 0 || p.C == 0) return true;
  if (p.n_blocks > 65535) return false;
  const dim3 gg((p.n_tok + kGateTok - 1) / kGateTok, p.n_blocks, (2 * p.n + kGateOut - 1) / kGateOut);
  SEQ_DISPATCH_T(bf16, lru_gates_kernel<T><<<gg, kGateThreads, 0, s>>>(p));
  const int cb = (p.C + kLruThreads - 1) / kLruThreads;
  if (p.max_runs <= 1) {
    SEQ_DISPATCH_T(bf16, lru_apply_kernel<T, false><<<dim3(cb, 1, R), kLruThreads, 0, s>>>(p));
    return true;
  }
  SEQ_DISPATCH_T(bf16, lru_reduce_kernel<T><<<dim3(cb, p.max_runs, R), kLruThreads, 0, s>>>(p));
  lru_carry_kernel<<<dim3(cb, 1, R), kLruThreads, 0, s>>>(p);
  SEQ_DISPATCH_T(bf16, lru_apply_kernel<T, true><<<dim3(cb, p.max_runs, R), kLruThreads, 0, s>>>(p));
  return true;
}

}  // namespace b200seq
