// Causal attention with logistic weights for packed prompts on sm_100a: tcgen05 MMAs with the scores and the output in TMEM,
// a TMA-fed K / V ring, two 128-row query tiles per CTA whose weight warpgroups alternate with the tensor core.
//
//   s_j = cap(q . k_j * scale) + bias_h, cap(z) = softcap tanh(z / softcap);   o = turn_back(sum_{j <= i} sigmoid(s_j) v_j)
//
// The weights are not normalised, so there is no running maximum and the accumulator is never rescaled: per key block the scores
// leave TMEM once, become weights in fp32 and return as the 16-bit A operand of the value product.  tanh and the logistic
// function are each one ex2 and one rcp.  The epilogue turns the pairs (i, i + D / 2) of a row (or (2 i, 2 i + 1)) back by the
// token's angles, read from a table, and drops the padding columns.
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

#include "b200_api.h"
#include "common.cuh"

namespace b200 {
namespace {

constexpr int kTQ = 128, kTK = 128;
constexpr float kLog2E = 1.4426950408889634f;
constexpr int kWaitLimit = 1 << 20;

__device__ int g_sigmoid_attn_error = 0;

__device__ __forceinline__ float ex2f(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcpf(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi, bool bf16) {
  if (bf16) return pack_bf16x2(lo, hi);
  __half2 h = __floats2half2_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&h);
}
// false: the wait ran out here, or another thread of the CTA gave up
__device__ __forceinline__ bool wait_bar(uint64_t* bar, uint32_t parity, volatile int* failed) {
  for (int i = 0; i < kWaitLimit; ++i) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((i & 255) == 255 && *failed) return false;
  }
  *failed = 1;
  return false;
}

struct SigParams {
  const int* cu;          // [R + 1] sequence boundaries
  const float* bias;      // [H] (nullptr: none)
  const float* table;     // [T, n_pairs, 2] cosine and sine of the turn (nullptr: nothing turns back)
  void* o;                // [T, H, dv]
  int H, G, dv, n_pairs, interleaved, is_bf16;
  float c_tanh;           // scale * 2 log2(e) / softcap; without a cap: -scale * log2(e)
  float two_cap;          // 2 softcap log2(e); 0: no cap
  float cap;              // softcap log2(e)
};

template <int D>
struct SigSmem {
  static constexpr int kDC = D / 64;                     // 128-byte column chunks of a row
  static constexpr int kTile = kTQ * 128 * kDC;
  static constexpr int kStages = 2;
  static constexpr int kKOff = 2 * kTile;                // two query tiles, then the K ring, then the V ring
  static constexpr int kVOff = kKOff + kStages * kTile;
  static constexpr int kBarOff = kVOff + kStages * kTile;
  static constexpr int kTotal = kBarOff + 256 + 1024;
};

template <int D, bool kCap>
__global__ void __launch_bounds__(384, 1)
sigmoid_attn_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                    const __grid_constant__ CUtensorMap tmap_v, const SigParams p) {
  using L = SigSmem<D>;
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
  uint64_t* o_done = bars + 13;       // 2
  uint64_t* drained = bars + 15;      // 1, failure path only
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 16);
  volatile int* failed = reinterpret_cast<volatile int*>(bars + 17);

  const int warp_idx = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int blk = n_blk - 1 - static_cast<int>(blockIdx.x);                    // the longest rows first
  const int h = blockIdx.y, hk = h / (p.H / p.G);
  const int q0[2] = {blk * 2 * kTQ, blk * 2 * kTQ + kTQ};
  const int nk[2] = {q0[0] / kTK + 1, q0[1] < len ? q0[1] / kTK + 1 : 0};      // key blocks of each tile
  const int nmax = max(nk[0], nk[1]);

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1); mbar_init(&p_ready[i], 128); mbar_init(&o_done[i], 1);
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
      const int n_tiles = nk[1] > 0 ? 2 : 1;
      mbar_arrive_expect_tx(q_full, n_tiles * L::kTile);
      for (int t = 0; t < n_tiles; ++t)
        for (int c = 0; c < L::kDC; ++c) tma_load_3d(&tmap_q, q_full, sQ + t * L::kTile + c * (kTQ * 128), c * 64, h, seq0 + q0[t]);
      int j = 0;
      for (; j < nmax; ++j) {
        const int st = j % L::kStages;
        const uint32_t ph = ((j / L::kStages) & 1) ^ 1;
        if (!wait_bar(&k_empty[st], ph, failed)) break;
        mbar_arrive_expect_tx(&k_full[st], L::kTile);
        for (int c = 0; c < L::kDC; ++c) tma_load_3d(&tmap_k, &k_full[st], sK + st * L::kTile + c * (kTK * 128), c * 64, hk, seq0 + j * kTK);
        if (!wait_bar(&v_empty[st], ph, failed)) { ++j; break; }
        mbar_arrive_expect_tx(&v_full[st], L::kTile);
        for (int c = 0; c < L::kDC; ++c) tma_load_3d(&tmap_v, &v_full[st], sV + st * L::kTile + c * (kTK * 128), c * 64, hk, seq0 + j * kTK);
      }
      if (*failed) {                                        // let the copies in flight land before the CTA ends
        volatile int never = 0;
        wait_bar(q_full, 0, &never);
        for (int b = max(0, j - L::kStages); b < j; ++b) {
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
        const uint32_t a0 = smem_u32(sQ + t * L::kTile), b0 = smem_u32(sK + (j % L::kStages) * L::kTile);
#pragma unroll
        for (int k = 0; k < D / 16; ++k) {
          const uint32_t off = (k >> 2) * (kTQ * 128) + (k & 3) * 32;
          umma_f16_ss(tmem_S + t * 128, make_smem_desc_sw128(a0 + off, 1024, 0), make_smem_desc_sw128(b0 + off, 1024, 0), idesc_s,
                      k != 0 ? 1u : 0u);
        }
        umma_commit(&s_full[t]);
      };
      auto issue_PV = [&](int t, int j) {
        const uint32_t b0 = smem_u32(sV + (j % L::kStages) * L::kTile);
#pragma unroll
        for (int k = 0; k < kTK / 16; ++k)                   // 16 keys per step: 8 packed columns of P; V is N-major
          umma_f16_ts(tmem_O + t * D, tmem_S + t * 128 + k * 8, make_smem_desc_sw128(b0 + k * 16 * 128, 1024, kTK * 128), idesc_o,
                      (j | k) != 0 ? 1u : 0u);
        if (j + 1 == nk[t]) umma_commit(&o_done[t]);
      };
      bool ok = wait_bar(q_full, 0, failed) && wait_bar(&k_full[0], 0, failed);
      if (ok) {
        tc_fence_after();
        issue_S(0, 0);
        if (nk[1] > 0) issue_S(1, 0);
        umma_commit(&k_empty[0]);
        for (int j = 0; j < nmax && ok; ++j) {
          const int nx = (j + 1) % L::kStages;
          ok = wait_bar(&v_full[j % L::kStages], (j / L::kStages) & 1, failed) &&
               (j + 1 >= nmax || wait_bar(&k_full[nx], ((j + 1) / L::kStages) & 1, failed));
          for (int t = 0; t < 2 && ok; ++t) {
            if (j >= nk[t]) continue;
            ok = wait_bar(&p_ready[t], j & 1, failed);
            if (!ok) break;
            tc_fence_after();
            issue_PV(t, j);
            if (j + 1 < nk[t]) issue_S(t, j + 1);
          }
          if (!ok) break;
          umma_commit(&v_empty[j % L::kStages]);
          if (j + 1 < nmax) umma_commit(&k_empty[nx]);
        }
      }
      if (!ok) {                                            // the MMAs in flight finish before TMEM is freed
        volatile int never = 0;
        umma_commit(drained);
        wait_bar(drained, 0, &never);
      }
    }
  } else if (warp_idx >= 4) {
    // ---------------------------------------------------------------- weights, epilogue
    const int t = (warp_idx - 4) >> 2, quad = warp_idx & 3;
    const int row = quad * 32 + lane, qrow = q0[t] + row;
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t tS = tmem_S + t * 128 + lane_addr, tO = tmem_O + t * D + lane_addr;
    const bool bf = p.is_bf16 != 0;
    const float bias = (p.bias != nullptr ? p.bias[h] : 0.f) * kLog2E;
    const float c1 = p.c_tanh, two_cap = p.two_cap, off = kCap ? -(p.cap + bias) : -bias;
    const int n = nk[t];
    bool ok = true;
    for (int j = 0; j < n && ok; ++j) {
      ok = __all_sync(0xffffffffu, wait_bar(&s_full[t], j & 1, failed));
      if (!ok) break;
      tc_fence_after();
      const int limit = qrow + 1 - j * kTK;                 // columns below it are visible
      const bool mask = j * kTK + kTK - 1 > q0[t];          // the diagonal block
      uint32_t v[2][32];
      tmem_ld_32x32(tS, v[0]);
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        tmem_ld_wait();
        if (c < 3) tmem_ld_32x32(tS + (c + 1) * 32, v[(c + 1) & 1]);
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          float w[2];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float s = __uint_as_float(v[c & 1][i + e]);
            float y;                                        // minus the score, times log2(e)
            if constexpr (kCap) y = fmaf(two_cap, rcpf(1.f + ex2f(s * c1)), off);
            else y = fmaf(s, c1, off);
            w[e] = rcpf(1.f + ex2f(y));
            if (mask && c * 32 + i + e >= limit) w[e] = 0.f;
          }
          pk[i >> 1] = pack2(w[0], w[1], bf);
        }
        // packed weights of chunk c -> columns [16 c, 16 c + 16); the scores they overwrite have been read
        tmem_st_32x16(tS + c * 16, pk);
      }
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_ready[t]);
    }
    if (n > 0 && ok) {
      ok = __all_sync(0xffffffffu, wait_bar(&o_done[t], 0, failed));
      if (ok) {
        tc_fence_after();
        const bool valid = qrow < len;
        const int64_t tok = seq0 + qrow;
        uint16_t* out = static_cast<uint16_t*>(p.o) + (tok * p.H + h) * p.dv;
        const float2* tab = p.table != nullptr ? reinterpret_cast<const float2*>(p.table) + tok * p.n_pairs : nullptr;
        auto put16 = [&](int c0, const uint32_t (&pk)[16], int n_cols) {     // 32 values at column c0, n_cols of them real
          if (!valid || n_cols <= 0) return;
          uint16_t* o = out + c0;
          if (n_cols >= 32 && (reinterpret_cast<uintptr_t>(o) & 15) == 0) {
#pragma unroll
            for (int u = 0; u < 4; ++u) *reinterpret_cast<uint4*>(o + u * 8) = make_uint4(pk[u * 4], pk[u * 4 + 1], pk[u * 4 + 2], pk[u * 4 + 3]);
          } else {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (i < n_cols) o[i] = static_cast<uint16_t>((i & 1) ? pk[i >> 1] >> 16 : pk[i >> 1] & 0xffffu);
          }
        };
        if (tab == nullptr || p.interleaved) {
#pragma unroll
          for (int c = 0; c < D / 32; ++c) {
            uint32_t v[32], pk[16];
            tmem_ld_32x32(tO + c * 32, v);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              float a = __uint_as_float(v[2 * i]), b = __uint_as_float(v[2 * i + 1]);
              if (tab != nullptr && valid && c * 16 + i < p.n_pairs) {
                const float2 cs = tab[c * 16 + i];
                const float x = a * cs.x + b * cs.y, z = b * cs.x - a * cs.y;
                a = x; b = z;
              }
              pk[i] = pack2(a, b, bf);
            }
            put16(c * 32, pk, p.dv - c * 32);
          }
        } else {
#pragma unroll
          for (int c = 0; c < D / 64; ++c) {                 // columns 32 c .. of the first half with those of the second half
            uint32_t va[32], vb[32], pa[16], pb[16];
            tmem_ld_32x32(tO + c * 32, va);
            tmem_ld_32x32(tO + D / 2 + c * 32, vb);
            tmem_ld_wait();
            const int left = p.n_pairs - c * 32;
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              float x[2], z[2];
#pragma unroll
              for (int e = 0; e < 2; ++e) {
                const float a = __uint_as_float(va[2 * i + e]), b = __uint_as_float(vb[2 * i + e]);
                float2 cs = make_float2(1.f, 0.f);
                if (valid && 2 * i + e < left) cs = tab[c * 32 + 2 * i + e];
                x[e] = a * cs.x + b * cs.y;
                z[e] = b * cs.x - a * cs.y;
              }
              pa[i] = pack2(x[0], x[1], bf);
              pb[i] = pack2(z[0], z[1], bf);
            }
            put16(c * 32, pa, left);
            put16(p.n_pairs + c * 32, pb, left);
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (threadIdx.x == 0 && *failed) atomicExch(&g_sigmoid_attn_error, 1);
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
thread_local std::string g_sig_error;

// [T, heads, D] contiguous: box 64 columns x 1 head x 128 tokens
bool make_map(CUtensorMap* map, const void* base, bool is_bf16, int D, int heads, int T) {
  ensure_cuda_context();
  EncodeFn fn = encode_fn();
  if (!fn) { g_sig_error = "cuTensorMapEncodeTiled unavailable"; return false; }
  cuuint64_t dims[3] = {static_cast<cuuint64_t>(D), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(T)};
  cuuint64_t strides[2] = {static_cast<cuuint64_t>(D) * 2, static_cast<cuuint64_t>(D) * heads * 2};
  cuuint32_t box[3] = {64, 1, 128};
  cuuint32_t estr[3] = {1, 1, 1};
  CUresult r = fn(map, is_bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 3, const_cast<void*>(base), dims, strides, box,
                  estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) { g_sig_error = "cuTensorMapEncodeTiled(3d) failed: code " + std::to_string(static_cast<int>(r)); return false; }
  return true;
}

template <int D, bool kCap>
int launch(const SigAttnArgs& a, const SigParams& p, cudaStream_t s) {
  CUtensorMap tq{}, tk{}, tv{};
  if (!make_map(&tq, a.q, a.is_bf16, D, a.H, a.n_tok) || !make_map(&tk, a.k, a.is_bf16, D, a.G, a.n_tok) ||
      !make_map(&tv, a.v, a.is_bf16, D, a.G, a.n_tok)) return -5;
  auto kern = sigmoid_attn_kernel<D, kCap>;
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SigSmem<D>::kTotal);
    if (e != cudaSuccess) { g_sig_error = std::string("cudaFuncSetAttribute: ") + cudaGetErrorString(e); return -10; }
    attr_set = true;
  }
  dim3 grid((a.max_len + 2 * kTQ - 1) / (2 * kTQ), a.H, a.n_seqs);
  kern<<<grid, 384, SigSmem<D>::kTotal, s>>>(tq, tk, tv, p);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) { g_sig_error = std::string("sigmoid_attn launch: ") + cudaGetErrorString(e); return -11; }
  return 0;
}

}  // namespace

const char* sigmoid_attn_last_error() { return g_sig_error.c_str(); }

int sigmoid_attn_status() {
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, g_sigmoid_attn_error, sizeof(int)) != cudaSuccess) return -1;
  return v;
}

int sigmoid_attn_fwd(const SigAttnArgs& a, cudaStream_t s) {
  if (a.d != 64 && a.d != 128) { g_sig_error = "padded head width must be 64 or 128"; return -1; }
  if (a.H % a.G != 0 || a.H > 65535 || a.n_seqs > 65535) { g_sig_error = "bad head or sequence count"; return -1; }
  if (a.dv > a.d || (a.table != nullptr && 2 * a.n_pairs > a.dv)) { g_sig_error = "bad value width"; return -1; }
  for (const void* ptr : {a.q, a.k, a.v})
    if (reinterpret_cast<uintptr_t>(ptr) % 16 != 0) { g_sig_error = "operands must be 16-byte aligned"; return -4; }
  if (a.n_tok == 0 || a.n_seqs == 0) return 0;
  SigParams p{};
  p.cu = a.cu; p.bias = a.bias; p.table = a.table; p.o = a.o;
  p.H = a.H; p.G = a.G; p.dv = a.dv; p.n_pairs = a.n_pairs; p.interleaved = a.interleaved; p.is_bf16 = a.is_bf16 ? 1 : 0;
  const bool cap = a.softcap > 0.f;
  p.cap = a.softcap * kLog2E; p.two_cap = 2.f * p.cap;
  p.c_tanh = cap ? a.scale * 2.f * kLog2E / a.softcap : -a.scale * kLog2E;
  if (a.d == 128) return cap ? launch<128, true>(a, p, s) : launch<128, false>(a, p, s);
  return cap ? launch<64, true>(a, p, s) : launch<64, false>(a, p, s);
}

}  // namespace b200
