// Sliding-window softmax attention for packed prompts on sm_100a: tcgen05 MMAs with the scores and the output in TMEM, a TMA-fed
// K / V ring, two 128-row query tiles per CTA whose softmax warpgroups alternate with the tensor core.
//
//   s_j = q_i . k_j * scale,  0 <= i - j < window;   o_i = sigmoid(g_i) * sum_j exp(s_j) v_j / (exp(sink_h) + sum_j exp(s_j))
//
// window 0: all earlier keys; the sink (a learned logit per head without a key) and the elementwise output gate are optional.  Keys are
// walked in blocks of 128 from the one that holds a tile's first visible key to the diagonal, so the work per row grows with
// the window, not with the position.  The two tiles of a CTA share the ring; a tile sits out the blocks it does not see.  The sink
// starts the running maximum and sum; the accumulator is rescaled only when the maximum has grown by more than 2^8.  The weights
// return to TMEM as the 16-bit A operand of the value product.
//
// Sequences lie one after another along the token axis; a CTA handles two query tiles of one head of one sequence.  Tiles that
// reach into the next sequence read its tokens (or zeros past the end) and mask them out.
// Every wait is bounded: a CTA whose wait runs out raises the error flag, lets its own copies and MMAs finish, frees its TMEM and
// returns.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <mutex>
#include <string>
#include <type_traits>

#include "b200_api.h"
#include "common.cuh"

namespace b200 {
namespace {

constexpr int kTQ = 128, kTK = 128;
constexpr float kLog2E = 1.4426950408889634f;
constexpr float kRescale = 8.0f;
constexpr int kWaitLimit = 1 << 20;

__device__ int g_window_attn_error = 0;

__device__ __forceinline__ float ex2f(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi, bool bf16) {
  if (bf16) return pack_bf16x2(lo, hi);
  __half2 h = __floats2half2_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&h);
}
__device__ __forceinline__ float2 unpack2(uint32_t v, bool bf16) {
  if (bf16) return unpack_bf16x2(v);
  return __half22float2(*reinterpret_cast<const __half2*>(&v));
}
__device__ __forceinline__ float from16(uint16_t v, bool bf16) { return unpack2(v, bf16).x; }
__device__ __forceinline__ float logistic(float x) { return 1.f / (1.f + __expf(-x)); }
// false: the wait ran out here, or another thread of the CTA gave up
__device__ __forceinline__ bool wait_bar(uint64_t* bar, uint32_t parity, volatile int* failed) {
  for (int i = 0; i < kWaitLimit; ++i) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((i & 255) == 255 && *failed) return false;
  }
  *failed = 1;
  return false;
}

struct WinParams {
  const int* cu;          // [R + 1] sequence boundaries
  const uint16_t* sink;   // [H] (nullptr: none)
  const uint16_t* gate;   // [T, H * dv] pre-activation, row stride ldg (nullptr: none)
  int64_t ldg;
  void* o;                // [T, H, dv]
  int H, G, dv, window, is_bf16;
  float scale_log2;       // scale * log2(e)
};

template <int D>
struct WinSmem {
  static constexpr int kDC = D / 64;                     // 128-byte column chunks of a row
  static constexpr int kTile = kTQ * 128 * kDC;
  static constexpr int kStages = 2;
  static constexpr int kKOff = 2 * kTile;                // two query tiles, then the K ring, then the V ring
  static constexpr int kVOff = kKOff + kStages * kTile;
  static constexpr int kBarOff = kVOff + kStages * kTile;
  static constexpr int kTotal = kBarOff + 256 + 1024;
};

template <int D>
__global__ void __launch_bounds__(384, 1)
window_attn_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                   const __grid_constant__ CUtensorMap tmap_v, const WinParams p) {
  using L = WinSmem<D>;
  const int r = blockIdx.z, seq0 = p.cu[r], len = p.cu[r + 1] - seq0;
  const int n_blk = (len + 2 * kTQ - 1) / (2 * kTQ);
  if (static_cast<int>(blockIdx.x) >= n_blk) return;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t *sQ = smem, *sK = smem + L::kKOff, *sV = smem + L::kVOff;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::kBarOff);
  uint64_t* q_full = bars;            // 1
  uint64_t* k_full = bars + 1;        // 2
  uint64_t* k_empty = bars + 3;       // 2
  uint64_t* v_full = bars + 5;        // 2
  uint64_t* v_empty = bars + 7;       // 2
  uint64_t* s_full = bars + 9;        // 2 (per query tile)
  uint64_t* p_ready = bars + 11;      // 2
  uint64_t* pv_done = bars + 13;      // 2
  uint64_t* drained = bars + 15;      // 1, failure path only
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 16);
  volatile int* failed = reinterpret_cast<volatile int*>(bars + 17);

  const int warp_idx = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int blk = n_blk - 1 - static_cast<int>(blockIdx.x);                    // the longest rows first
  const int h = blockIdx.y, hk = h / (p.H / p.G);
  const int q0[2] = {blk * 2 * kTQ, blk * 2 * kTQ + kTQ};
  // tile t works on key blocks lo[t] .. hi[t] - 1
  const int lo[2] = {p.window > 0 ? max(0, q0[0] - p.window + 1) / kTK : 0, p.window > 0 ? max(0, q0[1] - p.window + 1) / kTK : 0};
  const int hi[2] = {q0[0] / kTK + 1, q0[1] < len ? q0[1] / kTK + 1 : lo[1]};
  const int j_lo = lo[0], j_hi = max(hi[0], hi[1]);                            // lo[0] <= lo[1]

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1); mbar_init(&p_ready[i], 128); mbar_init(&pv_done[i], 1);
    }
    mbar_init(drained, 1);
    *failed = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmap_q); tma_prefetch_desc(&tmap_k); tma_prefetch_desc(&tmap_v);
  }
  if (warp_idx == 2) tmem_alloc<512>(tmem_slot);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_S = tmem_base;          // scores of tile t at column 128 t
  const uint32_t tmem_O = tmem_base + 256;    // output of tile t at column 256 + D t

  if (warp_idx == 0) {
    // ---------------------------------------------------------------- TMA producer
    if (lane == 0) {
      const int n_tiles = hi[1] > lo[1] ? 2 : 1;
      mbar_arrive_expect_tx(q_full, n_tiles * L::kTile);
      for (int t = 0; t < n_tiles; ++t)
        for (int c = 0; c < L::kDC; ++c) tma_load_3d(&tmap_q, q_full, sQ + t * L::kTile + c * (kTQ * 128), c * 64, h, seq0 + q0[t]);
      int j = j_lo;
      for (; j < j_hi; ++j) {
        const int n = j - j_lo, st = n % L::kStages;
        const uint32_t ph = ((n / L::kStages) & 1) ^ 1;
        if (!wait_bar(&k_empty[st], ph, failed)) break;
        mbar_arrive_expect_tx(&k_full[st], L::kTile);
        for (int c = 0; c < L::kDC; ++c) tma_load_3d(&tmap_k, &k_full[st], sK + st * L::kTile + c * (kTK * 128), c * 64, hk, seq0 + j * kTK);
        if (!wait_bar(&v_empty[st], ph, failed)) break;
        mbar_arrive_expect_tx(&v_full[st], L::kTile);
        for (int c = 0; c < L::kDC; ++c) tma_load_3d(&tmap_v, &v_full[st], sV + st * L::kTile + c * (kTK * 128), c * 64, hk, seq0 + j * kTK);
      }
      if (*failed) {                                        // let the copies in flight land before the CTA ends
        volatile int never = 0;
        wait_bar(q_full, 0, &never);
        const int n = j - j_lo;
        for (int b = max(0, n - L::kStages); b <= n && b < j_hi - j_lo; ++b) {
          wait_bar(&k_full[b % L::kStages], (b / L::kStages) & 1, &never);
          wait_bar(&v_full[b % L::kStages], (b / L::kStages) & 1, &never);
        }
      }
    }
  } else if (warp_idx == 1) {
    // ---------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      const uint32_t idesc_s = make_idesc_f16(p.is_bf16 != 0, kTQ, kTK, false, false);
      const uint32_t idesc_o = make_idesc_f16(p.is_bf16 != 0, kTQ, D, false, true);
      auto issue_S = [&](int t, int j) {
        const uint32_t a0 = smem_u32(sQ + t * L::kTile), b0 = smem_u32(sK + ((j - j_lo) % L::kStages) * L::kTile);
#pragma unroll
        for (int k = 0; k < D / 16; ++k) {
          const uint32_t off = (k >> 2) * (kTQ * 128) + (k & 3) * 32;
          umma_f16_ss(tmem_S + t * 128, make_smem_desc_sw128(a0 + off, 1024, 0), make_smem_desc_sw128(b0 + off, 1024, 0), idesc_s,
                      k != 0 ? 1u : 0u);
        }
        umma_commit(&s_full[t]);
      };
      auto issue_PV = [&](int t, int j) {
        const uint32_t b0 = smem_u32(sV + ((j - j_lo) % L::kStages) * L::kTile);
#pragma unroll
        for (int k = 0; k < kTK / 16; ++k)                   // 16 keys per step: 8 packed columns of P; V is N-major
          umma_f16_ts(tmem_O + t * D, tmem_S + t * 128 + k * 8, make_smem_desc_sw128(b0 + k * 16 * 128, 1024, kTK * 128), idesc_o,
                      (j > lo[t] || k != 0) ? 1u : 0u);
        umma_commit(&pv_done[t]);
      };
      bool ok = wait_bar(q_full, 0, failed) && wait_bar(&k_full[0], 0, failed);
      if (ok) {
        tc_fence_after();
        for (int t = 0; t < 2; ++t)
          if (lo[t] == j_lo && hi[t] > lo[t]) issue_S(t, j_lo);
        umma_commit(&k_empty[0]);
        for (int j = j_lo; j < j_hi && ok; ++j) {
          const int n = j - j_lo, nx = (n + 1) % L::kStages;
          ok = wait_bar(&v_full[n % L::kStages], (n / L::kStages) & 1, failed) &&
               (j + 1 >= j_hi || wait_bar(&k_full[nx], ((n + 1) / L::kStages) & 1, failed));
          for (int t = 0; t < 2 && ok; ++t) {
            if (j >= lo[t] && j < hi[t]) {
              ok = wait_bar(&p_ready[t], (j - lo[t]) & 1, failed);
              if (!ok) break;
              tc_fence_after();
              issue_PV(t, j);
            }
            if (j + 1 >= lo[t] && j + 1 < hi[t]) issue_S(t, j + 1);
          }
          if (!ok) break;
          umma_commit(&v_empty[n % L::kStages]);
          if (j + 1 < j_hi) umma_commit(&k_empty[nx]);
        }
      }
      if (!ok) {                                            // the MMAs in flight finish before TMEM is freed
        volatile int never = 0;
        umma_commit(drained);
        wait_bar(drained, 0, &never);
      }
    }
  } else if (warp_idx >= 4) {
    // ---------------------------------------------------------------- softmax, epilogue
    const int t = (warp_idx - 4) >> 2, quad = warp_idx & 3;
    const int row = quad * 32 + lane, qrow = q0[t] + row;
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t tS = tmem_S + t * 128 + lane_addr, tO = tmem_O + t * D + lane_addr;
    const bool bf = p.is_bf16 != 0;
    const float sc = p.scale_log2;
    const int from = lo[t], n = hi[t] - lo[t];
    float m = -INFINITY, l = 0.f;                           // running maximum (exp2 domain) and sum
    if (p.sink != nullptr) {
      m = from16(p.sink[h], bf) * kLog2E;
      l = m > -INFINITY ? 1.f : 0.f;
    }
    bool ok = true;

    // one key block: the row maximum first, then the weights; first_col .. limit - 1 are the visible columns
    auto block = [&](int i, int first_col, int limit, auto masked_tag) {
      constexpr bool kMasked = decltype(masked_tag)::value;
      float mx = -INFINITY;
      {
        uint32_t v[2][32];
        tmem_ld_32x32(tS, v[0]);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          tmem_ld_wait();
          if (c < 3) tmem_ld_32x32(tS + (c + 1) * 32, v[(c + 1) & 1]);
#pragma unroll
          for (int e = 0; e < 32; ++e) {
            float x = __uint_as_float(v[c & 1][e]) * sc;
            if (kMasked && (c * 32 + e >= limit || c * 32 + e < first_col)) x = -INFINITY;
            mx = fmaxf(mx, x);
          }
        }
      }
      const float m_new = fmaxf(m, mx);
      const bool grow = m_new > m + kRescale;               // also true for the first visible key (m = -inf)
      const float m_cur = grow ? m_new : m;
      const float alpha = grow ? ex2f(m - m_cur) : 1.f;
      const float m_use = m_cur == -INFINITY ? 0.f : m_cur; // nothing visible yet: keep the arithmetic finite
      if (i > 0) {
        ok = __all_sync(0xffffffffu, wait_bar(&pv_done[t], (i - 1) & 1, failed));
        if (!ok) return;
        tc_fence_after();
        if (__any_sync(0xffffffffu, grow)) {
#pragma unroll
          for (int c = 0; c < D / 32; ++c) {
            uint32_t v[32];
            tmem_ld_32x32(tO + c * 32, v);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 32; ++e) v[e] = __float_as_uint(__uint_as_float(v[e]) * alpha);
            tmem_st_32x32(tO + c * 32, v);
          }
          tmem_st_wait();
        }
      }
      l *= alpha;
      float rs0 = 0.f, rs1 = 0.f;
      {
        uint32_t v[2][32];
        tmem_ld_32x32(tS, v[0]);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          tmem_ld_wait();
          if (c < 3) tmem_ld_32x32(tS + (c + 1) * 32, v[(c + 1) & 1]);
          uint32_t pk[16];
#pragma unroll
          for (int e = 0; e < 32; e += 2) {
            float w0 = ex2f(fmaf(__uint_as_float(v[c & 1][e]), sc, -m_use));
            float w1 = ex2f(fmaf(__uint_as_float(v[c & 1][e + 1]), sc, -m_use));
            if (kMasked) {
              if (c * 32 + e >= limit || c * 32 + e < first_col) w0 = 0.f;
              if (c * 32 + e + 1 >= limit || c * 32 + e + 1 < first_col) w1 = 0.f;
            }
            rs0 += w0;
            rs1 += w1;
            pk[e >> 1] = pack2(w0, w1, bf);
          }
          // packed weights of chunk c -> columns [16 c, 16 c + 16); the scores they overwrite have been read
          tmem_st_32x16(tS + c * 16, pk);
        }
      }
      l += rs0 + rs1;
      m = m_cur;
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_ready[t]);
    };

    for (int i = 0; i < n && ok; ++i) {
      ok = __all_sync(0xffffffffu, wait_bar(&s_full[t], i & 1, failed));
      if (!ok) break;
      tc_fence_after();
      const int kbase = (from + i) * kTK;
      const int limit = qrow + 1 - kbase, first_col = p.window > 0 ? qrow + 1 - p.window - kbase : -kTK;
      // the diagonal block, or one that some row of the tile sees only from the middle on
      const bool mask = kbase + kTK - 1 > q0[t] || (p.window > 0 && kbase < q0[t] + kTQ - p.window);
      if (mask) block(i, first_col, limit, std::true_type{});
      else block(i, first_col, limit, std::false_type{});
    }
    if (n > 0 && ok) {
      ok = __all_sync(0xffffffffu, wait_bar(&pv_done[t], (n - 1) & 1, failed));
      if (ok) {
        tc_fence_after();
        const bool valid = qrow < len;
        const float inv_l = l > 0.f ? 1.f / l : 0.f;
        const int64_t tok = seq0 + qrow;
        uint16_t* out = static_cast<uint16_t*>(p.o) + (tok * p.H + h) * p.dv;
        const uint16_t* gate = p.gate != nullptr ? p.gate + tok * p.ldg + h * p.dv : nullptr;
        const bool wide = p.dv % 8 == 0 && (reinterpret_cast<uintptr_t>(p.o) & 15) == 0 &&
                          (p.gate == nullptr || (p.ldg % 8 == 0 && (reinterpret_cast<uintptr_t>(p.gate) & 15) == 0));
#pragma unroll
        for (int c = 0; c < D / 32; ++c) {
          uint32_t v[32];
          tmem_ld_32x32(tO + c * 32, v);
          tmem_ld_wait();
          if (!valid) continue;
          if (wide) {
#pragma unroll
            for (int u = 0; u < 4; ++u) {
              const int col = c * 32 + u * 8;
              if (col >= p.dv) continue;
              float f[8];
#pragma unroll
              for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(v[u * 8 + e]) * inv_l;
              if (gate != nullptr) {
                const uint4 g = *reinterpret_cast<const uint4*>(gate + col);
                const uint32_t gw[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                  const float2 x = unpack2(gw[e], bf);
                  f[2 * e] *= logistic(x.x);
                  f[2 * e + 1] *= logistic(x.y);
                }
              }
              *reinterpret_cast<uint4*>(out + col) = make_uint4(pack2(f[0], f[1], bf), pack2(f[2], f[3], bf), pack2(f[4], f[5], bf), pack2(f[6], f[7], bf));
            }
          } else {
#pragma unroll
            for (int e = 0; e < 32; ++e) {
              const int col = c * 32 + e;
              if (col < p.dv) {
                float f = __uint_as_float(v[e]) * inv_l;
                if (gate != nullptr) f *= logistic(from16(gate[col], bf));
                out[col] = static_cast<uint16_t>(pack2(f, 0.f, bf) & 0xffffu);
              }
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (threadIdx.x == 0 && *failed) atomicExch(&g_window_attn_error, 1);
  if (warp_idx == 2) tmem_dealloc<512>(tmem_base);
}

// ------------------------------------------------------------------------------------ host side
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
thread_local std::string g_win_error;

// [T, heads, D] contiguous: box 64 columns x 1 head x 128 tokens
bool make_map(CUtensorMap* map, const void* base, bool is_bf16, int D, int heads, int T) {
  ensure_cuda_context();
  EncodeFn fn = encode_fn();
  if (!fn) { g_win_error = "cuTensorMapEncodeTiled unavailable"; return false; }
  cuuint64_t dims[3] = {static_cast<cuuint64_t>(D), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(T)};
  cuuint64_t strides[2] = {static_cast<cuuint64_t>(D) * 2, static_cast<cuuint64_t>(D) * heads * 2};
  cuuint32_t box[3] = {64, 1, 128};
  cuuint32_t estr[3] = {1, 1, 1};
  CUresult r = fn(map, is_bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 3, const_cast<void*>(base), dims, strides, box,
                  estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) { g_win_error = "cuTensorMapEncodeTiled(3d) failed: code " + std::to_string(static_cast<int>(r)); return false; }
  return true;
}

template <int D>
int launch(const WinAttnArgs& a, const WinParams& p, cudaStream_t s) {
  CUtensorMap tq{}, tk{}, tv{};
  if (!make_map(&tq, a.q, a.is_bf16, D, a.H, a.n_tok) || !make_map(&tk, a.k, a.is_bf16, D, a.G, a.n_tok) ||
      !make_map(&tv, a.v, a.is_bf16, D, a.G, a.n_tok)) return -5;
  auto kern = window_attn_kernel<D>;
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, WinSmem<D>::kTotal);
    if (e != cudaSuccess) { g_win_error = std::string("cudaFuncSetAttribute: ") + cudaGetErrorString(e); return -10; }
    attr_set = true;
  }
  dim3 grid((a.max_len + 2 * kTQ - 1) / (2 * kTQ), a.H, a.n_seqs);
  kern<<<grid, 384, WinSmem<D>::kTotal, s>>>(tq, tk, tv, p);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) { g_win_error = std::string("window_attn launch: ") + cudaGetErrorString(e); return -11; }
  return 0;
}

}  // namespace

const char* window_attn_last_error() { return g_win_error.c_str(); }

int window_attn_status() {
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_window_attn_error, sizeof(int)) != cudaSuccess) return -1;
  return v;
}

int window_attn_fwd(const WinAttnArgs& a, cudaStream_t s) {
  if (a.d != 64 && a.d != 128) { g_win_error = "padded head width must be 64 or 128"; return -1; }
  if (a.G < 1 || a.H % a.G != 0 || a.H > 65535 || a.n_seqs > 65535) { g_win_error = "bad head or sequence count"; return -1; }
  if (a.dv > a.d || a.window < 0 || !(a.scale > 0.f)) { g_win_error = "bad value width, window or scale"; return -1; }
  for (const void* ptr : {a.q, a.k, a.v})
    if (reinterpret_cast<uintptr_t>(ptr) % 16 != 0) { g_win_error = "operands must be 16-byte aligned"; return -4; }
  if (a.n_tok == 0 || a.n_seqs == 0) return 0;
  WinParams p{};
  p.cu = a.cu; p.sink = static_cast<const uint16_t*>(a.sink); p.gate = static_cast<const uint16_t*>(a.gate); p.ldg = a.ldg; p.o = a.o;
  p.H = a.H; p.G = a.G; p.dv = a.dv; p.window = a.window; p.is_bf16 = a.is_bf16 ? 1 : 0;
  p.scale_log2 = a.scale * kLog2E;
  return a.d == 128 ? launch<128>(a, p, s) : launch<64>(a, p, s);
}

}  // namespace b200
