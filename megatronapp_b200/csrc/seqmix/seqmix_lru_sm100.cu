// Real-gated linear recurrent unit for 16-bit prompts on sm_100a: the block-diagonal gates run on tcgen05 and feed the recurrence
// straight from TMEM.
//
// A CTA owns 128 channels of one gate block and a chunk of kChunk tokens of one sequence.  TMA brings the two gate matrices'
// rows (K-major, zero-filled past the block) and the chunk's inputs; two chains of MMAs leave the pre-activations of the
// recurrence and the input gate in TMEM as [channel][token].  A thread then owns one channel (a TMEM lane) and walks its tokens in
// registers: gates, decay, what the token writes.  The recurrence is linear, so it takes two such kernels: the first reduces every
// chunk to (P, Q) with S_end = P S_begin + Q, a small one carries the state over a sequence's chunks, the second walks every
// chunk again from its S_begin and writes S * gelu_tanh(y_pre).
// Every wait is bounded: when one runs out the CTA raises the error flag, lets its own copies and MMAs finish, frees its TMEM and
// returns.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <mutex>

#include "../common.cuh"
#include "seq_lru.cuh"
#include "seqmix_api.h"

namespace b200seq {

namespace {

using namespace b200;

constexpr int kChunk = 128, kChan = 128;                   // tokens and channels of a CTA
constexpr int kWaitLimit = 1 << 20;
constexpr float kLog2E = 1.4426950408889634f;

__device__ int g_lru_error = 0;

__device__ __forceinline__ bool wait_bar(uint64_t* bar, uint32_t parity) {
  for (int i = 0; i < kWaitLimit; ++i)
    if (mbar_try_wait(bar, parity)) return true;
  return false;
}
__device__ __forceinline__ void tma_load_4d(const void* tmap, uint64_t* bar, void* smem_dst, int32_t c0, int32_t c1, int32_t c2, int32_t c3) {
  asm volatile(
      "cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6}], [%2];"
      ::"r"(smem_u32(smem_dst)), "l"(tmap), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2), "r"(c3)
      : "memory");
}
__device__ __forceinline__ float ex2f(float x) { float y; asm("ex2.approx.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float rcpf(float x) { float y; asm("rcp.approx.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float sqrtf_(float x) { float y; asm("sqrt.approx.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// as dev::lru_gates with one ex2 / rcp per logistic function; 1 - a^2 by its series (in 2 log a) where a is near one
__device__ __forceinline__ void gates_fast(float r_pre, float i_pre, float u, float rate, float* a, float* put) {
  const float r = rcpf(1.f + ex2f(-kLog2E * r_pre)), i = rcpf(1.f + ex2f(-kLog2E * i_pre));
  const float la = -rate * r, x = 2.f * la;
  const float av = ex2f(kLog2E * la);
  const float series = -x * fmaf(x, fmaf(x, fmaf(x, fmaf(x, fmaf(x, fmaf(x, 1.f / 5040.f, 1.f / 720.f), 1.f / 120.f), 1.f / 24.f), 1.f / 6.f), 0.5f), 1.f);
  const float left = x > -0.25f ? series : fmaf(-av, av, 1.f);
  *a = av;
  *put = sqrtf_(left) * i * u;
}
__device__ __forceinline__ float gelu_fast(float z) {      // z / (1 + exp(-2 y)) with y the tanh's argument
  return z * rcpf(1.f + ex2f(-2.f * kLog2E * 0.7978845608028654f * fmaf(0.044715f * z * z, z, z)));
}

struct ChunkArgs {
  LruArgs p;
  int k_chunks, k_steps;                                   // 64-wide pieces and 16-wide MMA steps of the block's width
};

// grid (chunks, blocks x channel tiles, sequences)
template <bool APPLY>
__global__ void __launch_bounds__(128)
lru_chunk_kernel(const __grid_constant__ CUtensorMap map_u, const __grid_constant__ CUtensorMap map_w, const ChunkArgs args) {
  const LruArgs& p = args.p;
  const int seq = blockIdx.z, lo = p.cu[seq] + blockIdx.x * kChunk, n_tok = min(p.cu[seq + 1] - lo, kChunk);
  if (n_tok <= 0) return;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int tile = args.k_chunks * (128 * 128);            // bytes of a [128 rows x width] operand
  uint8_t *sU = smem, *sR = smem + tile, *sI = smem + 2 * tile;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + 3 * tile);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2);
  volatile int* failed = reinterpret_cast<volatile int*>(bars + 3);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tiles = (p.n + kChan - 1) / kChan, blk = blockIdx.y / tiles, o0 = (blockIdx.y % tiles) * kChan;

  if (threadIdx.x == 0) {
    mbar_init(&bars[0], 1);
    mbar_init(&bars[1], 1);
    *failed = 0;
    mbar_fence_init();
  }
  if (warp == 0) tmem_alloc<256>(tmem_slot);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;                        // recurrence gate at columns 0 .., input gate at 128 ..
  if (threadIdx.x == 0) {
    mbar_arrive_expect_tx(&bars[0], 3 * tile);
    for (int c = 0; c < args.k_chunks; ++c) {
      tma_load_3d(&map_u, &bars[0], sU + c * (128 * 128), c * 64, blk, lo);
      tma_load_4d(&map_w, &bars[0], sR + c * (128 * 128), c * 64, o0, 0, blk);
      tma_load_4d(&map_w, &bars[0], sI + c * (128 * 128), c * 64, o0, 1, blk);
    }
    if (wait_bar(&bars[0], 0)) {
      tc_fence_after();
      const uint32_t idesc = make_idesc_f16(true, kChan, kChunk, false, false);
      const uint32_t u0 = smem_u32(sU), r0 = smem_u32(sR), i0 = smem_u32(sI);
      for (int k = 0; k < args.k_steps; ++k) {
        const uint32_t off = (k >> 2) * (128 * 128) + (k & 3) * 32;
        const uint64_t du = make_smem_desc_sw128(u0 + off, 1024, 0);
        umma_f16_ss(tmem, make_smem_desc_sw128(r0 + off, 1024, 0), du, idesc, k != 0 ? 1u : 0u);
        umma_f16_ss(tmem + 128, make_smem_desc_sw128(i0 + off, 1024, 0), du, idesc, k != 0 ? 1u : 0u);
      }
      umma_commit(&bars[1]);
    } else {
      *failed = 1;
      wait_bar(&bars[0], 0);                               // the copies in flight, once more
      umma_commit(&bars[1]);                               // nothing was issued: the other threads are released at once
    }
  }
  if (!wait_bar(&bars[0], 0) || !wait_bar(&bars[1], 0)) *failed = 1;         // every thread reads the inputs from shared memory
  __syncthreads();
  if (!*failed) {
    tc_fence_after();
    const int o = o0 + threadIdx.x;                        // output channel within the block
    const bool live = o < p.n;
    const int c = blk * p.n + min(o, p.n - 1);
    const __nv_bfloat16* bias = static_cast<const __nv_bfloat16*>(p.bias) + static_cast<int64_t>(blk) * 2 * p.n + (c - blk * p.n);
    const float br = __bfloat162float(bias[0]), bi = __bfloat162float(bias[p.n]);
    const float rate = p.decay_scale * dev::softplusf_(__bfloat162float(static_cast<const __nv_bfloat16*>(p.lam)[c]));
    float* ws = p.ws + ((static_cast<int64_t>(seq) * p.max_runs + blockIdx.x) * p.C + c) * 2;
    float P = 1.f, S = APPLY ? ws[0] : 0.f;
    const uint32_t row = tmem + (static_cast<uint32_t>(warp * 32) << 16);
    const int uc = c - blk * p.n;
    const uint8_t* su = sU + (uc >> 6) * (128 * 128) + (uc & 7) * 2;
    const int unit = (uc & 63) >> 3;
    const __nv_bfloat16* yp = static_cast<const __nv_bfloat16*>(p.y_pre) + (p.y_pre != nullptr ? static_cast<int64_t>(lo) * p.ldy + c : 0);
    __nv_bfloat16* y = static_cast<__nv_bfloat16*>(p.y) + static_cast<int64_t>(lo) * p.C + c;
    __nv_bfloat16 ynext[16];                                       // one batch ahead of its use
    auto fetch_y = [&](int t0) {
#pragma unroll
      for (int j = 0; j < 16; ++j) ynext[j] = yp[static_cast<int64_t>(min(t0 + j, n_tok - 1)) * p.ldy];
    };
    if (APPLY && p.y_pre != nullptr) fetch_y(0);
    for (int t0 = 0; t0 < n_tok; t0 += 16) {               // the same trip count for the whole CTA: TMEM loads are warp-wide
      uint32_t vr[16], vi[16];
      tmem_ld_32x16(row + t0, vr);
      tmem_ld_32x16(row + 128 + t0, vi);
      float yv[16];
      if (APPLY && p.y_pre != nullptr) {
#pragma unroll
        for (int j = 0; j < 16; ++j) yv[j] = __bfloat162float(ynext[j]);
        fetch_y(t0 + 16);
      }
      tmem_ld_wait();
      // the sixteen tokens' gates are independent of each other and of the state; tokens past the end keep the state as it is
      float a[16], put[16];
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        const int t = t0 + j;
        const float u = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(su + t * 128 + ((unit ^ (t & 7)) << 4)));
        gates_fast(__uint_as_float(vr[j]) + br, __uint_as_float(vi[j]) + bi, u, rate, &a[j], &put[j]);
        if (t >= n_tok) { a[j] = 1.f; put[j] = 0.f; }
      }
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        if constexpr (!APPLY) P *= a[j];
        S = fmaf(a[j], S, put[j]);
        put[j] = S;
      }
      if constexpr (APPLY) {
        if (p.y_pre != nullptr) {
#pragma unroll
          for (int j = 0; j < 16; ++j) put[j] *= gelu_fast(yv[j]);
        }
#pragma unroll
        for (int j = 0; j < 16; ++j)
          if (live && t0 + j < n_tok) y[static_cast<int64_t>(t0 + j) * p.C] = __float2bfloat16_rn(put[j]);
      }
    }
    if (!APPLY && live) { ws[0] = P; ws[1] = S; }
  } else if (threadIdx.x == 0) {
    atomicExch(&g_lru_error, 1);
    wait_bar(&bars[1], 0);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc<256>(tmem);
}

__global__ void __launch_bounds__(128) lru_chunk_carry_kernel(LruArgs p) {
  const int c = blockIdx.x * 128 + threadIdx.x, r = blockIdx.y;
  const int n = p.cu[r + 1] - p.cu[r];
  if (c >= p.C || n <= 0) return;
  float* state = p.state + static_cast<int64_t>(p.rows[r]) * p.C + c;
  float S = *state;
  float2* ws = reinterpret_cast<float2*>(p.ws) + static_cast<int64_t>(r) * p.max_runs * p.C + c;
  const int chunks = (n + kChunk - 1) / kChunk;
  for (int y0 = 0; y0 < chunks; y0 += 8) {                 // the loads of eight chunks go out before the chain
    float2 v[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = y0 + j < chunks ? ws[static_cast<int64_t>(y0 + j) * p.C] : make_float2(1.f, 0.f);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (y0 + j < chunks) {
        ws[static_cast<int64_t>(y0 + j) * p.C].x = S;      // the chunk's starting state
        S = fmaf(v[j].x, S, v[j].y);
      }
    }
  }
  *state = S;
}

typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                             const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeFn encode_fn() {
  static EncodeFn fn = nullptr;
  static std::once_flag once;
  std::call_once(once, [] {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &qres) == cudaSuccess && qres == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<EncodeFn>(ptr);
  });
  return fn;
}
bool encode(CUtensorMap* map, int rank, const void* base, const cuuint64_t* dims, const cuuint64_t* strides, const cuuint32_t* box) {
  EncodeFn fn = encode_fn();
  const cuuint32_t one[4] = {1, 1, 1, 1};
  return fn != nullptr && fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, static_cast<cuuint32_t>(rank), const_cast<void*>(base), dims, strides, box, one,
                             CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                             CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

}  // namespace

int lru_chunks(int max_len) { return (max_len + kChunk - 1) / kChunk; }

bool rglru_chunked_supported(const LruArgs& p, int max_len) {
  return max_len >= 32 && p.n % 8 == 0 && p.n <= 256 && p.ldu % 8 == 0 && reinterpret_cast<uintptr_t>(p.u) % 16 == 0 &&
         reinterpret_cast<uintptr_t>(p.w) % 16 == 0 && static_cast<int64_t>(p.n_blocks) * ((p.n + kChan - 1) / kChan) <= 65535;
}

int rglru_chunked_status() {
  int v = 0;
  return cudaMemcpyFromSymbol(&v, g_lru_error, sizeof(int)) == cudaSuccess ? v : -1;
}

bool rglru_scan_chunked(const LruArgs& p, int R, cudaStream_t s) {
  if (R == 0 || p.n_tok == 0) return true;
  if (R > 65535) return false;
  cudaFree(nullptr);                                       // the driver entry point needs a context
  CUtensorMap mu{}, mw{};
  const cuuint64_t n = p.n, B = p.n_blocks;
  const cuuint64_t du[3] = {n, B, static_cast<cuuint64_t>(p.n_tok)}, ds[2] = {n * 2, static_cast<cuuint64_t>(p.ldu) * 2};
  const cuuint32_t bu[3] = {64, 1, kChunk};
  const cuuint64_t wd[4] = {n, n, 2, B}, wst[3] = {n * 2, n * n * 2, 2 * n * n * 2};
  const cuuint32_t bw[4] = {64, kChan, 1, 1};
  if (!encode(&mu, 3, p.u, du, ds, bu) || !encode(&mw, 4, p.w, wd, wst, bw)) return false;
  ChunkArgs a{p, (p.n + 63) / 64, (p.n + 15) / 16};
  const int smem = 3 * a.k_chunks * (128 * 128) + 64 + 1024;
  static std::once_flag once;
  std::call_once(once, [] {
    const int most = 3 * 4 * (128 * 128) + 64 + 1024;
    cudaFuncSetAttribute(lru_chunk_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
    cudaFuncSetAttribute(lru_chunk_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
  });
  const dim3 grid(p.max_runs, p.n_blocks * ((p.n + kChan - 1) / kChan), R);
  lru_chunk_kernel<false><<<grid, 128, smem, s>>>(mu, mw, a);
  lru_chunk_carry_kernel<<<dim3((p.C + 127) / 128, R), 128, 0, s>>>(p);
  lru_chunk_kernel<true><<<grid, 128, smem, s>>>(mu, mw, a);
  return true;
}

}  // namespace b200seq
