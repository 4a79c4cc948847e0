// PyTorch bindings of the sequence-mixing kernels (pybind11 module megatronapp_b200._C_seq).
#include <torch/extension.h>
#include <algorithm>
#include <atomic>
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>

#include "seqmix_api.h"

using torch::Tensor;

namespace {

std::atomic<int64_t> g_launches{0};
inline cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }
inline void count(int n = 1) { g_launches.fetch_add(n, std::memory_order_relaxed); }

bool act_is_bf16(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
  TORCH_CHECK(t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat, name, " must be bf16 or fp32, got ", t.scalar_type());
  return t.scalar_type() == at::kBFloat16;
}
void check_f32(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous(), name, " must be a contiguous fp32 CUDA tensor");
}
void check_i32(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kInt && t.is_contiguous(), name, " must be a contiguous int32 CUDA tensor");
}
void check_rows(const Tensor& t, const char* name) {   // [T, ...] with contiguous trailing dims and a free row stride
  TORCH_CHECK(t.dim() == 3 && t.stride(2) == 1 && t.stride(1) == t.size(2), name, " must be [T, heads, dim] with contiguous heads");
}
void check_last_error(const char* what) {
  cudaError_t e = cudaGetLastError();
  TORCH_CHECK(e == cudaSuccess, what, ": ", cudaGetErrorString(e));
}

void add_rms_norm(Tensor x, c10::optional<Tensor> delta, const Tensor& w, Tensor y, double eps, double w_off) {
  check_f32(x, "x");
  const bool bf16 = act_is_bf16(y, "y");
  TORCH_CHECK(x.dim() == 2 && y.is_contiguous() && y.sizes() == x.sizes(), "x / y must be [rows, cols]");
  TORCH_CHECK(w.scalar_type() == y.scalar_type() && w.is_contiguous() && w.numel() == x.size(1), "weight must match y's dtype and cols");
  TORCH_CHECK(x.size(1) * sizeof(float) <= 48 * 1024, "row too wide");
  const void* d = nullptr;
  if (delta.has_value() && delta->defined()) {
    TORCH_CHECK(delta->scalar_type() == y.scalar_type() && delta->is_contiguous() && delta->sizes() == x.sizes(),
                "delta must be contiguous, shaped like x, in y's dtype");
    d = delta->data_ptr();
  }
  c10::cuda::CUDAGuard g(x.device());
  b200seq::add_rms_norm(x.data_ptr<float>(), d, w.data_ptr(), y.data_ptr(), static_cast<int>(x.size(0)), static_cast<int>(x.size(1)),
                        static_cast<float>(eps), static_cast<float>(w_off), bf16, cur_stream());
  count(); check_last_error("add_rms_norm");
}

void gated_head_rms_norm(const Tensor& o, c10::optional<Tensor> w_opt, c10::optional<Tensor> gate, Tensor y, double eps, bool silu) {
  check_f32(o, "o");
  TORCH_CHECK(o.dim() == 3, "o must be [T, H, dv]");
  const bool bf16 = act_is_bf16(y, "y");
  const int T = static_cast<int>(o.size(0)), H = static_cast<int>(o.size(1)), dv = static_cast<int>(o.size(2));
  TORCH_CHECK(y.is_contiguous() && y.numel() == o.numel(), "y must be [T, H * dv]");
  const void* wp = nullptr;
  bool per_head = false;
  if (w_opt.has_value() && w_opt->defined()) {
    const Tensor& w = *w_opt;
    TORCH_CHECK(w.is_cuda() && w.scalar_type() == y.scalar_type() && w.is_contiguous() && (w.numel() == dv || w.numel() == H * dv), "bad weight");
    wp = w.data_ptr(); per_head = w.numel() != dv || H == 1;
  }
  const void* gp = nullptr;
  int64_t ldg = 0;
  if (gate.has_value() && gate->defined()) {
    TORCH_CHECK(gate->is_cuda() && gate->scalar_type() == y.scalar_type() && gate->dim() == 2 && gate->stride(1) == 1 && gate->size(0) == T &&
                gate->size(1) == static_cast<int64_t>(H) * dv, "gate must be [T, H * dv] with unit inner stride");
    gp = gate->data_ptr(); ldg = gate->stride(0);
  }
  c10::cuda::CUDAGuard g(o.device());
  b200seq::gated_head_rms_norm(o.data_ptr<float>(), wp, gp, ldg, y.data_ptr(), T, H, dv, per_head, eps, silu, bf16, cur_stream());
  count(); check_last_error("gated_head_rms_norm");
}

void causal_conv(const Tensor& x, const Tensor& w, c10::optional<Tensor> bias, const Tensor& cu, const Tensor& rows,
                 const Tensor& tok_seq, Tensor window, Tensor y, int64_t max_len, bool silu, bool residual) {
  const bool bf16 = act_is_bf16(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1, "x must be [T, C] with unit inner stride");
  const int T = static_cast<int>(x.size(0)), C = static_cast<int>(x.size(1)), taps = static_cast<int>(w.size(1));
  TORCH_CHECK(w.scalar_type() == x.scalar_type() && w.is_contiguous() && w.size(0) == C, "bad conv weight");
  TORCH_CHECK(y.scalar_type() == x.scalar_type() && y.is_contiguous() && y.sizes() == x.sizes(), "bad y");
  TORCH_CHECK(window.scalar_type() == x.scalar_type() && window.is_contiguous() && window.dim() == 3 && window.size(1) == taps - 1 &&
              window.size(2) == C, "window must be [rows, taps - 1, C]");
  check_i32(cu, "cu"); check_i32(rows, "rows"); check_i32(tok_seq, "tok_seq");
  TORCH_CHECK(tok_seq.numel() == T && cu.numel() == rows.numel() + 1, "bad packed-batch tensors");
  const void* bp = nullptr;
  if (bias.has_value() && bias->defined()) {
    TORCH_CHECK(bias->scalar_type() == x.scalar_type() && bias->is_contiguous() && bias->numel() == C, "bad conv bias");
    bp = bias->data_ptr();
  }
  c10::cuda::CUDAGuard g(x.device());
  b200seq::causal_conv_silu(x.data_ptr(), x.stride(0), w.data_ptr(), bp, cu.data_ptr<int>(), rows.data_ptr<int>(), tok_seq.data_ptr<int>(),
                            window.data_ptr(), y.data_ptr(), T, static_cast<int>(rows.numel()), C, taps, static_cast<int>(max_len), silu, residual, bf16,
                            cur_stream());
  count(2); check_last_error("causal_conv_silu");
}

void delta_rule_scan(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& log_decay, const Tensor& beta, const Tensor& cu,
                     const Tensor& rows, Tensor state, Tensor out, double unit_eps, double q_scale, int64_t max_len) {
  const bool bf16 = act_is_bf16(q, "q");
  TORCH_CHECK(k.scalar_type() == q.scalar_type() && v.scalar_type() == q.scalar_type(), "q / k / v dtypes differ");
  check_rows(q, "q"); check_rows(k, "k"); check_rows(v, "v");
  check_f32(log_decay, "log_decay"); check_f32(beta, "beta"); check_f32(state, "state"); check_f32(out, "out");
  check_i32(cu, "cu"); check_i32(rows, "rows");
  b200seq::DeltaArgs p{};
  p.q = q.data_ptr(); p.k = k.data_ptr(); p.v = v.data_ptr();
  p.ldq = q.stride(0); p.ldk = k.stride(0); p.ldv = v.stride(0);
  p.H = static_cast<int>(v.size(1)); p.KH = static_cast<int>(q.size(1)); p.d = static_cast<int>(q.size(2)); p.dv = static_cast<int>(v.size(2));
  TORCH_CHECK(p.H % p.KH == 0 && k.size(1) == p.KH && k.size(2) == p.d, "bad head layout");
  p.decay_per_head = log_decay.numel() == q.size(0) * p.H && (log_decay.dim() == 2 || p.d == 1) ? 1 : 0;
  TORCH_CHECK((p.decay_per_head || log_decay.numel() == q.size(0) * p.H * p.d) && beta.numel() == q.size(0) * p.H, "bad decay / beta shape");
  TORCH_CHECK(state.dim() == 4 && state.size(1) == p.H && state.size(2) == p.d && state.size(3) == p.dv, "bad state shape");
  TORCH_CHECK(out.numel() == q.size(0) * p.H * p.dv, "bad out shape");
  p.log_decay = log_decay.data_ptr<float>(); p.beta = beta.data_ptr<float>();
  p.cu = cu.data_ptr<int>(); p.rows = rows.data_ptr<int>();
  p.state = state.data_ptr<float>(); p.out = out.data_ptr<float>();
  p.unit_eps = static_cast<float>(unit_eps); p.q_scale = static_cast<float>(q_scale);
  p.max_len = max_len > 0 ? static_cast<int>(max_len) : (1 << 30);
  c10::cuda::CUDAGuard g(q.device());
  TORCH_CHECK(b200seq::delta_rule_scan(p, static_cast<int>(rows.numel()), bf16, cur_stream()), "delta_rule_scan: key dim ", p.d,
              " above the largest kernel instance (256)");
  count(); check_last_error("delta_rule_scan");
}

void mlstm_scan(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& log_i, const Tensor& log_f, const Tensor& cu,
                const Tensor& rows, Tensor state, Tensor norm_state, Tensor max_state, Tensor out, double q_scale, double denom_eps,
                int64_t max_len) {
  const bool bf16 = act_is_bf16(q, "q");
  TORCH_CHECK(k.scalar_type() == q.scalar_type() && v.scalar_type() == q.scalar_type(), "q / k / v dtypes differ");
  check_rows(q, "q"); check_rows(k, "k"); check_rows(v, "v");
  check_f32(log_i, "log_i"); check_f32(log_f, "log_f"); check_f32(state, "state"); check_f32(norm_state, "norm_state");
  check_f32(max_state, "max_state"); check_f32(out, "out");
  check_i32(cu, "cu"); check_i32(rows, "rows");
  b200seq::MlstmArgs p{};
  p.q = q.data_ptr(); p.k = k.data_ptr(); p.v = v.data_ptr();
  p.ldq = q.stride(0); p.ldk = k.stride(0); p.ldv = v.stride(0);
  p.H = static_cast<int>(v.size(1)); p.d = static_cast<int>(q.size(2)); p.dv = static_cast<int>(v.size(2));
  TORCH_CHECK(q.size(1) == p.H && k.size(1) == p.H && k.size(2) == p.d, "bad head layout");
  TORCH_CHECK(log_i.numel() == q.size(0) * p.H && log_f.numel() == q.size(0) * p.H, "bad gate shape");
  TORCH_CHECK(state.dim() == 4 && state.size(1) == p.H && state.size(2) == p.d && state.size(3) == p.dv, "bad state shape");
  TORCH_CHECK(norm_state.numel() == state.size(0) * p.H * p.d && max_state.numel() == state.size(0) * p.H, "bad n / m shape");
  TORCH_CHECK(out.numel() == q.size(0) * p.H * p.dv, "bad out shape");
  p.log_i = log_i.data_ptr<float>(); p.log_f = log_f.data_ptr<float>();
  p.cu = cu.data_ptr<int>(); p.rows = rows.data_ptr<int>();
  p.state = state.data_ptr<float>(); p.norm_state = norm_state.data_ptr<float>(); p.max_state = max_state.data_ptr<float>();
  p.out = out.data_ptr<float>();
  p.q_scale = static_cast<float>(q_scale); p.denom_eps = static_cast<float>(denom_eps);
  p.max_len = max_len > 0 ? static_cast<int>(max_len) : (1 << 30);
  c10::cuda::CUDAGuard g(q.device());
  TORCH_CHECK(b200seq::mlstm_scan(p, static_cast<int>(rows.numel()), bf16, cur_stream()), "mlstm_scan: key dim ", p.d,
              " above the largest kernel instance (256)");
  count(); check_last_error("mlstm_scan");
}

const void* opt_ptr(const c10::optional<Tensor>& t) { return (t.has_value() && t->defined()) ? t->data_ptr() : nullptr; }
void check_act2(const Tensor& t, const Tensor& like, const char* name) {   // [T, C], unit inner stride, free row stride
  TORCH_CHECK(t.is_cuda() && t.dim() == 2 && t.stride(1) == 1 && t.scalar_type() == like.scalar_type(), name,
              " must be a [T, C] CUDA tensor with unit inner stride in the activation dtype");
}

void latent_attention_paged(const Tensor& q, c10::optional<Tensor> q_rot, const Tensor& cache, const Tensor& block_table, const Tensor& tok_req,
                            const Tensor& tok_len, c10::optional<Tensor> gate, Tensor out, int64_t block_size, double scale, int64_t max_len,
                            int64_t window, c10::optional<Tensor> sink) {
  const bool bf16 = act_is_bf16(q, "q_lat");
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous(), "q_lat must be contiguous [T, H, r]");
  b200seq::LatentAttnArgs p{};
  if (opt_ptr(q_rot) != nullptr) {
    TORCH_CHECK(q_rot->scalar_type() == q.scalar_type() && q_rot->dim() == 3 && q_rot->is_contiguous() && q_rot->size(0) == q.size(0) &&
                q_rot->size(1) == q.size(1), "q_rot must be contiguous [T, H, n] in q_lat's dtype");
    p.q_rot = q_rot->data_ptr(); p.n_rot = static_cast<int>(q_rot->size(2));
  }
  TORCH_CHECK(cache.scalar_type() == q.scalar_type() && cache.dim() == 2 && cache.is_contiguous() && cache.size(1) == q.size(2) + p.n_rot,
              "cache must be [slots, r (+ n)] in q_lat's dtype");
  check_i32(block_table, "block_table"); check_i32(tok_req, "tok_req"); check_i32(tok_len, "tok_len"); check_f32(out, "out");
  TORCH_CHECK(block_table.dim() == 2 && tok_req.numel() == q.size(0) && tok_len.numel() == q.size(0) && out.numel() == q.numel(),
              "bad shapes");
  if (opt_ptr(gate) != nullptr) {
    check_act2(*gate, q, "gate");
    TORCH_CHECK(gate->size(0) == q.size(0) && gate->size(1) == q.size(1), "gate must be [T, H]");
    p.gate = gate->data_ptr(); p.ldg = gate->stride(0);
  }
  if (opt_ptr(sink) != nullptr) {
    TORCH_CHECK(sink->is_cuda() && sink->scalar_type() == q.scalar_type() && sink->is_contiguous() && sink->numel() == q.size(1),
                "sink must be [H] in q_lat's dtype");
    p.sink = sink->data_ptr();
  }
  p.window = static_cast<int>(window);
  if (window > 0) max_len = std::min(max_len, window);
  p.q = q.data_ptr(); p.cache = cache.data_ptr();
  p.block_table = block_table.data_ptr<int>(); p.tok_req = tok_req.data_ptr<int>(); p.tok_len = tok_len.data_ptr<int>();
  p.out = out.data_ptr<float>();
  p.H = static_cast<int>(q.size(1)); p.r = static_cast<int>(q.size(2)); p.block_size = static_cast<int>(block_size);
  p.max_blocks = static_cast<int>(block_table.size(1)); p.scale = static_cast<float>(scale);
  c10::cuda::CUDAGuard g(q.device());
  p.n_splits = b200seq::latent_attention_splits(p.H, p.r + p.n_rot, static_cast<int>(q.size(0)), static_cast<int>(max_len));
  const int64_t vec = 16 / static_cast<int64_t>(cache.element_size());
  p.vec_ok = ((p.r + p.n_rot) % vec == 0 && reinterpret_cast<uintptr_t>(cache.data_ptr()) % 16 == 0) ? 1 : 0;
  Tensor ws;
  if (p.n_splits > 1) {
    ws = torch::empty({q.size(0), q.size(1), p.n_splits, q.size(2) + 2}, out.options());
    p.ws = ws.data_ptr<float>();
  }
  TORCH_CHECK(b200seq::latent_attention_paged(p, static_cast<int>(q.size(0)), bf16, cur_stream()), "latent_attention_paged: rank ", p.r + p.n_rot,
              " above the largest kernel instance (1024)");
  count(p.n_splits > 1 ? 2 : 1); check_last_error("latent_attention_paged");
}

void group_limited_router(const Tensor& logits, c10::optional<Tensor> correction, Tensor probs, Tensor rmap, int64_t topk, int64_t groups,
                          int64_t keep, bool renorm, bool sigmoid, bool top2, double scale) {
  check_f32(logits, "logits"); check_f32(probs, "probs");
  TORCH_CHECK(logits.dim() == 2 && probs.sizes() == logits.sizes() && rmap.sizes() == logits.sizes() && rmap.scalar_type() == at::kBool &&
              rmap.is_contiguous(), "bad shapes");
  const float* cp = nullptr;
  if (opt_ptr(correction) != nullptr) {
    check_f32(*correction, "correction");
    TORCH_CHECK(correction->numel() == logits.size(1), "correction must be [experts]");
    cp = correction->data_ptr<float>();
  }
  c10::cuda::CUDAGuard g(logits.device());
  TORCH_CHECK(b200seq::group_limited_router(logits.data_ptr<float>(), cp, probs.data_ptr<float>(), rmap.data_ptr<bool>(),
                                            static_cast<int>(logits.size(0)), static_cast<int>(logits.size(1)), static_cast<int>(topk),
                                            static_cast<int>(groups), static_cast<int>(keep), renorm, sigmoid, top2, static_cast<float>(scale),
                                            cur_stream()),
              "group_limited_router: unsupported sizes (experts ", logits.size(1), ", groups ", groups, ", top ", topk, ")");
  count(); check_last_error("group_limited_router");
}


// ---- side-by-side mixer, minGRU, clamped gated activation ------------------------------------------------------------------
void norm_add(Tensor x, const Tensor& a, c10::optional<Tensor> b, c10::optional<Tensor> wa, c10::optional<Tensor> wb,
              c10::optional<Tensor> w, Tensor y, double eps, double w_off, c10::optional<Tensor> extra, c10::optional<Tensor> next_w) {
  check_f32(x, "x");
  const bool bf16 = act_is_bf16(y, "y");
  TORCH_CHECK(x.dim() == 2 && y.is_contiguous() && y.sizes() == x.sizes(), "x / y must be [rows, cols]");
  TORCH_CHECK(a.is_cuda() && a.scalar_type() == y.scalar_type() && a.is_contiguous() && a.sizes() == x.sizes(), "a must be contiguous, shaped like x");
  TORCH_CHECK(x.size(1) * sizeof(float) <= 48 * 1024, "row too wide");
  auto vec = [&](const c10::optional<Tensor>& t, const char* name) -> const void* {
    if (!t.has_value() || !t->defined()) return nullptr;
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == y.scalar_type() && t->is_contiguous() && t->numel() == x.size(1), name,
                " must be a contiguous [cols] tensor in y's dtype");
    return t->data_ptr();
  };
  const bool two = b.has_value() && b->defined();
  if (two) {
    TORCH_CHECK(b->is_cuda() && b->scalar_type() == y.scalar_type() && b->is_contiguous() && b->sizes() == x.sizes(), "b must be shaped like a");
    TORCH_CHECK(vec(wa, "weight_a") != nullptr && vec(wb, "weight_b") != nullptr, "two branches need their norm weights");
  }
  const void* ex = nullptr;
  if (extra.has_value() && extra->defined()) {
    TORCH_CHECK(extra->is_cuda() && extra->scalar_type() == y.scalar_type() && extra->is_contiguous() && extra->sizes() == x.sizes(),
                "extra must be contiguous, shaped like x, in y's dtype");
    ex = extra->data_ptr();
  }
  c10::cuda::CUDAGuard g(x.device());
  b200seq::norm_add(x.data_ptr<float>(), a.data_ptr(), two ? b->data_ptr() : nullptr, two ? vec(wa, "weight_a") : nullptr,
                    two ? vec(wb, "weight_b") : nullptr, vec(w, "weight"), y.data_ptr(), static_cast<int>(x.size(0)),
                    static_cast<int>(x.size(1)), static_cast<float>(eps), static_cast<float>(w_off), ex, vec(next_w, "next_weight"), bf16,
                    cur_stream());
  count(); check_last_error("norm_add");
}

void retention_scan(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& decay, c10::optional<Tensor> positions,
                    c10::optional<Tensor> inv_freq, const Tensor& cu, const Tensor& rows, Tensor state, Tensor out, double k_scale,
                    int64_t max_len) {
  const bool bf16 = act_is_bf16(q, "q");
  TORCH_CHECK(k.scalar_type() == q.scalar_type() && v.scalar_type() == q.scalar_type(), "q / k / v dtypes differ");
  check_rows(q, "q"); check_rows(k, "k"); check_rows(v, "v");
  check_f32(decay, "decay"); check_f32(state, "state"); check_f32(out, "out");
  check_i32(cu, "cu"); check_i32(rows, "rows");
  b200seq::RetentionArgs p{};
  p.q = q.data_ptr(); p.k = k.data_ptr(); p.v = v.data_ptr();
  p.ldq = q.stride(0); p.ldk = k.stride(0); p.ldv = v.stride(0);
  p.H = static_cast<int>(v.size(1)); p.d = static_cast<int>(q.size(2)); p.dv = static_cast<int>(v.size(2));
  TORCH_CHECK(q.size(1) == p.H && k.size(1) == p.H && k.size(2) == p.d && v.size(0) == q.size(0) && k.size(0) == q.size(0), "bad head layout");
  TORCH_CHECK(decay.numel() == p.H, "decay must be [H]");
  TORCH_CHECK(state.dim() == 4 && state.size(1) == p.H && state.size(2) == p.d && state.size(3) == p.dv, "bad state shape");
  TORCH_CHECK(out.numel() == q.size(0) * p.H * p.dv, "bad out shape");
  if (inv_freq.has_value() && inv_freq->defined() && inv_freq->numel() > 0) {
    check_f32(*inv_freq, "inv_freq");
    p.n_rot = static_cast<int>(inv_freq->numel());
    TORCH_CHECK(2 * p.n_rot <= p.d, "more rotated dimensions than the head has");
    TORCH_CHECK(positions.has_value() && positions->is_cuda() && positions->scalar_type() == at::kLong && positions->is_contiguous() &&
                positions->numel() == q.size(0), "positions must be a contiguous int64 [T]");
    p.inv_freq = inv_freq->data_ptr<float>(); p.positions = positions->data_ptr<int64_t>();
  }
  p.decay = decay.data_ptr<float>();
  p.cu = cu.data_ptr<int>(); p.rows = rows.data_ptr<int>();
  p.state = state.data_ptr<float>(); p.out = out.data_ptr<float>();
  p.k_scale = static_cast<float>(k_scale);
  p.max_len = max_len > 0 ? static_cast<int>(max_len) : (1 << 30);
  c10::cuda::CUDAGuard g(q.device());
  TORCH_CHECK(b200seq::retention_scan(p, static_cast<int>(rows.numel()), bf16, cur_stream()), "retention_scan: key dim ", p.d,
              " above the largest kernel instance (256)");
  count(); check_last_error("retention_scan");
}

void poly_norm(const Tensor& z, const Tensor& coef, Tensor y, double eps) {
  const bool bf16 = act_is_bf16(z, "z");
  check_act2(z, z, "z"); check_f32(coef, "coef");
  TORCH_CHECK(coef.numel() == 4, "coef must hold four numbers");
  TORCH_CHECK(y.scalar_type() == z.scalar_type() && y.is_contiguous() && y.sizes() == z.sizes(), "bad y");
  c10::cuda::CUDAGuard g(z.device());
  TORCH_CHECK(b200seq::poly_norm(z.data_ptr(), z.stride(0), coef.data_ptr<float>(), y.data_ptr(), z.size(0), static_cast<int>(z.size(1)),
                                 static_cast<float>(eps), bf16, cur_stream()), "poly_norm: row too wide");
  count(); check_last_error("poly_norm");
}

void decay_gates(const Tensor& a, const Tensor& b, const Tensor& A_log, const Tensor& dt_bias, Tensor log_decay, Tensor beta) {
  const bool bf16 = act_is_bf16(a, "a");
  check_act2(a, a, "a"); check_act2(b, a, "b");
  check_f32(log_decay, "log_decay"); check_f32(beta, "beta");
  const int64_t rows = a.size(0);
  const int C = static_cast<int>(a.size(1)), H = static_cast<int>(b.size(1));
  TORCH_CHECK(b.size(0) == rows && H > 0 && C % H == 0, "a must be [T, C] and b [T, H] with C a multiple of H");
  TORCH_CHECK(A_log.is_cuda() && A_log.scalar_type() == a.scalar_type() && A_log.is_contiguous() && A_log.numel() == H &&
              dt_bias.is_cuda() && dt_bias.scalar_type() == a.scalar_type() && dt_bias.is_contiguous() && dt_bias.numel() == C, "bad A_log / dt_bias");
  TORCH_CHECK(log_decay.numel() == rows * C && beta.numel() == rows * H, "bad output shapes");
  c10::cuda::CUDAGuard g(a.device());
  b200seq::decay_gates(a.data_ptr(), a.stride(0), b.data_ptr(), b.stride(0), A_log.data_ptr(), dt_bias.data_ptr(), log_decay.data_ptr<float>(),
                       beta.data_ptr<float>(), rows, C, H, bf16, cur_stream());
  count(); check_last_error("decay_gates");
}

void gelu_mul(const Tensor& gt, const Tensor& e, Tensor y) {
  const bool bf16 = act_is_bf16(gt, "g");
  check_act2(gt, gt, "g"); check_act2(e, gt, "e");
  TORCH_CHECK(e.sizes() == gt.sizes() && y.scalar_type() == gt.scalar_type() && y.is_contiguous() && y.sizes() == gt.sizes(), "bad e / y");
  c10::cuda::CUDAGuard g(gt.device());
  b200seq::gelu_mul(gt.data_ptr(), gt.stride(0), e.data_ptr(), e.stride(0), y.data_ptr(), gt.size(0), static_cast<int>(gt.size(1)), bf16,
                    cur_stream());
  count(); check_last_error("gelu_mul");
}

void norm_rope(const Tensor& q, const Tensor& k, const Tensor& wq, const Tensor& wk, const Tensor& positions, const Tensor& inv_freq,
               Tensor q_out, Tensor k_out, int64_t head_dim, int64_t rot, double eps) {
  const bool bf16 = act_is_bf16(q, "q");
  check_act2(q, q, "q"); check_act2(k, q, "k");
  check_f32(inv_freq, "inv_freq");
  TORCH_CHECK(positions.is_cuda() && positions.scalar_type() == at::kLong && positions.is_contiguous() && positions.numel() == q.size(0),
              "positions must be a contiguous int64 [T]");
  TORCH_CHECK(rot % 2 == 0 && rot <= head_dim && inv_freq.numel() * 2 == rot, "rot must be even, at most head_dim, with rot / 2 frequencies");
  TORCH_CHECK(q.size(1) % head_dim == 0 && k.size(1) % head_dim == 0 && k.size(0) == q.size(0), "bad q / k shape");
  TORCH_CHECK(wq.scalar_type() == q.scalar_type() && wk.scalar_type() == q.scalar_type() && wq.is_contiguous() && wk.is_contiguous() &&
              wq.numel() == q.size(1) && wk.numel() == k.size(1), "bad norm weights");
  TORCH_CHECK(q_out.scalar_type() == q.scalar_type() && k_out.scalar_type() == q.scalar_type() && q_out.is_contiguous() &&
              k_out.is_contiguous() && q_out.numel() == q.numel() && k_out.numel() == k.numel(), "bad outputs");
  TORCH_CHECK((std::max(q.size(1), k.size(1)) + 1 + rot) * sizeof(float) <= 48 * 1024, "projection too wide");
  b200seq::NormRopeArgs p{};
  p.q = q.data_ptr(); p.k = k.data_ptr(); p.ldq = q.stride(0); p.ldk = k.stride(0);
  p.wq = wq.data_ptr(); p.wk = wk.data_ptr(); p.positions = positions.data_ptr<int64_t>(); p.inv_freq = inv_freq.data_ptr<float>();
  p.q_out = q_out.data_ptr(); p.k_out = k_out.data_ptr();
  p.q_ch = static_cast<int>(q.size(1)); p.k_ch = static_cast<int>(k.size(1)); p.head_dim = static_cast<int>(head_dim);
  p.rot = static_cast<int>(rot); p.eps = static_cast<float>(eps);
  c10::cuda::CUDAGuard g(q.device());
  b200seq::norm_rope(p, static_cast<int>(q.size(0)), bf16, cur_stream());
  count(); check_last_error("norm_rope");
}

void mixed_attention_paged(const Tensor& q, const Tensor& kcache, const Tensor& vcache, const Tensor& block_table, const Tensor& tok_req,
                           const Tensor& tok_len, c10::optional<Tensor> talk, c10::optional<Tensor> gate, Tensor out, int64_t block_size,
                           double scale, int64_t max_len, bool force_generic) {
  const bool bf16 = act_is_bf16(q, "q");
  check_rows(q, "q");
  TORCH_CHECK(kcache.scalar_type() == q.scalar_type() && vcache.scalar_type() == q.scalar_type() && kcache.dim() == 3 && vcache.dim() == 3 &&
              kcache.is_contiguous() && vcache.is_contiguous() && kcache.size(2) == q.size(2) && vcache.size(1) == kcache.size(1),
              "caches must be contiguous [slots, G, d] / [slots, G, dv] in q's dtype");
  check_i32(block_table, "block_table"); check_i32(tok_req, "tok_req"); check_i32(tok_len, "tok_len");
  b200seq::MixAttnArgs p{};
  p.H = static_cast<int>(q.size(1)); p.G = static_cast<int>(kcache.size(1)); p.d = static_cast<int>(q.size(2));
  p.dv = static_cast<int>(vcache.size(2));
  TORCH_CHECK(block_table.dim() == 2 && tok_req.numel() == q.size(0) && tok_len.numel() == q.size(0), "bad packed-batch tensors");
  TORCH_CHECK(out.scalar_type() == q.scalar_type() && out.is_contiguous() && out.numel() == q.size(0) * p.H * p.dv, "bad out");
  p.q = q.data_ptr(); p.ldq = q.stride(0); p.kcache = kcache.data_ptr(); p.vcache = vcache.data_ptr();
  p.block_table = block_table.data_ptr<int>(); p.tok_req = tok_req.data_ptr<int>(); p.tok_len = tok_len.data_ptr<int>();
  if (talk.has_value() && talk->defined()) {
    check_f32(*talk, "talk");
    TORCH_CHECK(talk->numel() == static_cast<int64_t>(p.H) * p.H, "talk must be [H, H]");
    p.talk = talk->data_ptr<float>();
  }
  if (gate.has_value() && gate->defined()) {
    check_act2(*gate, q, "gate");
    TORCH_CHECK(gate->size(0) == q.size(0) && gate->size(1) == p.H * p.dv, "gate must be [T, H * dv]");
    p.gate = gate->data_ptr(); p.ldg = gate->stride(0);
  }
  p.out = out.data_ptr();
  p.block_size = static_cast<int>(block_size); p.max_blocks = static_cast<int>(block_table.size(1)); p.scale = static_cast<float>(scale);
  c10::cuda::CUDAGuard g(q.device());
  p.n_splits = b200seq::mixed_attention_splits(static_cast<int>(q.size(0)), static_cast<int>(max_len));
  p.query_block = static_cast<int>(q.size(0) / std::max<int64_t>(1, block_table.size(0)));
  p.force_generic = force_generic ? 1 : 0;
  Tensor ws1, ws2;
  if (p.n_splits > 1) {
    auto o32 = q.options().dtype(at::kFloat);
    ws1 = torch::empty({q.size(0), p.n_splits, p.H, 2}, o32);
    ws2 = torch::empty({q.size(0), p.n_splits, static_cast<int64_t>(p.H) * p.dv}, o32);
    p.ws_stats = ws1.data_ptr<float>(); p.ws_acc = ws2.data_ptr<float>();
  }
  TORCH_CHECK(b200seq::mixed_attention_paged(p, static_cast<int>(q.size(0)), bf16, cur_stream()),
              "mixed_attention_paged: no kernel instance for heads ", p.H, " / ", p.G, ", dims ", p.d, " / ", p.dv);
  count(p.n_splits > 1 ? 3 : 1); check_last_error("mixed_attention_paged");
}

void gen_delta_scan(const Tensor& r, const Tensor& k, const Tensor& v, const Tensor& w_pre, const Tensor& a_pre, c10::optional<Tensor> w_bias,
                    const Tensor& cu, const Tensor& rows, Tensor state, Tensor out, double decay_scale, double unit_eps,
                    int64_t max_len) {
  const bool bf16 = act_is_bf16(r, "r");
  check_rows(r, "r"); check_rows(k, "k"); check_rows(v, "v");
  check_act2(w_pre, r, "w_pre"); check_act2(a_pre, r, "a_pre");
  TORCH_CHECK(k.scalar_type() == r.scalar_type() && v.scalar_type() == r.scalar_type(), "r / k / v dtypes differ");
  check_f32(state, "state"); check_f32(out, "out"); check_i32(cu, "cu"); check_i32(rows, "rows");
  b200seq::GenDeltaArgs p{};
  p.H = static_cast<int>(r.size(1)); p.d = static_cast<int>(r.size(2)); p.dv = static_cast<int>(v.size(2));
  TORCH_CHECK(k.size(1) == p.H && k.size(2) == p.d && v.size(1) == p.H, "bad head layout");
  TORCH_CHECK(w_pre.size(0) == r.size(0) && a_pre.size(0) == r.size(0) && w_pre.size(1) == p.H * p.d && a_pre.size(1) == p.H * p.d,
              "decay / removal pre-activations must be [T, H * d]");
  TORCH_CHECK(state.dim() == 4 && state.size(1) == p.H && state.size(2) == p.d && state.size(3) == p.dv, "bad state shape");
  TORCH_CHECK(out.numel() == r.size(0) * p.H * p.dv, "bad out shape");
  if (w_bias.has_value() && w_bias->defined()) {
    TORCH_CHECK(w_bias->scalar_type() == r.scalar_type() && w_bias->is_contiguous() && w_bias->numel() == p.H * p.d, "bad decay bias");
    p.w_bias = w_bias->data_ptr();
  }
  p.r = r.data_ptr(); p.k = k.data_ptr(); p.v = v.data_ptr(); p.w_pre = w_pre.data_ptr(); p.a_pre = a_pre.data_ptr();
  p.ldr = r.stride(0); p.ldk = k.stride(0); p.ldv = v.stride(0); p.ldw = w_pre.stride(0); p.lda = a_pre.stride(0);
  p.cu = cu.data_ptr<int>(); p.rows = rows.data_ptr<int>(); p.state = state.data_ptr<float>(); p.out = out.data_ptr<float>();
  p.decay_scale = static_cast<float>(decay_scale); p.unit_eps = static_cast<float>(unit_eps);
  p.max_len = max_len > 0 ? static_cast<int>(max_len) : (1 << 30);
  c10::cuda::CUDAGuard g(r.device());
  TORCH_CHECK(b200seq::gen_delta_scan(p, static_cast<int>(rows.numel()), bf16, cur_stream()), "gen_delta_scan: key dim ", p.d,
              " above the largest kernel instance (256)");
  count(); check_last_error("gen_delta_scan");
}

void mingru_scan(const Tensor& z_pre, const Tensor& u_pre, const Tensor& g_pre, const Tensor& cu, const Tensor& rows, Tensor state, Tensor y,
                 int64_t max_len) {
  const bool bf16 = act_is_bf16(z_pre, "z_pre");
  check_act2(z_pre, z_pre, "z_pre"); check_act2(u_pre, z_pre, "u_pre"); check_act2(g_pre, z_pre, "g_pre");
  check_f32(state, "state"); check_i32(cu, "cu"); check_i32(rows, "rows");
  b200seq::MinGruArgs p{};
  p.C = static_cast<int>(z_pre.size(1));
  TORCH_CHECK(u_pre.sizes() == z_pre.sizes() && g_pre.sizes() == z_pre.sizes() && state.dim() == 2 && state.size(1) == p.C, "bad shapes");
  TORCH_CHECK(y.scalar_type() == z_pre.scalar_type() && y.is_contiguous() && y.sizes() == z_pre.sizes(), "bad y");
  p.z_pre = z_pre.data_ptr(); p.u_pre = u_pre.data_ptr(); p.g_pre = g_pre.data_ptr();
  p.ldz = z_pre.stride(0); p.ldu = u_pre.stride(0); p.ldg = g_pre.stride(0);
  p.cu = cu.data_ptr<int>(); p.rows = rows.data_ptr<int>(); p.state = state.data_ptr<float>(); p.y = y.data_ptr();
  c10::cuda::CUDAGuard g(z_pre.device());
  const int R = static_cast<int>(rows.numel());
  p.max_runs = b200seq::mingru_runs(static_cast<int>(max_len));
  Tensor ws;
  if (p.max_runs > 1) {
    ws = torch::empty({R, p.max_runs, p.C, 2}, state.options());
    p.ws = ws.data_ptr<float>();
  }
  b200seq::mingru_scan(p, R, bf16, cur_stream());
  count(p.max_runs > 1 ? 3 : 1); check_last_error("mingru_scan");
}

void clamped_glu(const Tensor& x, Tensor y, double limit, double alpha, double shift) {
  const bool bf16 = act_is_bf16(x, "x");
  check_act2(x, x, "x");
  TORCH_CHECK(x.size(1) % 2 == 0 && y.scalar_type() == x.scalar_type() && y.is_contiguous() && y.dim() == 2 && y.size(0) == x.size(0) &&
              y.size(1) * 2 == x.size(1), "x must be [T, 2 F], y [T, F]");
  c10::cuda::CUDAGuard g(x.device());
  b200seq::clamped_glu(x.data_ptr(), x.stride(0), y.data_ptr(), x.size(0), static_cast<int>(y.size(1)), static_cast<float>(limit),
                       static_cast<float>(alpha), static_cast<float>(shift), bf16, cur_stream());
  count(); check_last_error("clamped_glu");
}



void stream_mix_norm(Tensor x, c10::optional<Tensor> a, c10::optional<Tensor> b, c10::optional<Tensor> bias_a, c10::optional<Tensor> ls,
                     double scale_a, double scale_b, c10::optional<Tensor> mix, c10::optional<Tensor> outc, c10::optional<Tensor> inp,
                     c10::optional<Tensor> w, c10::optional<Tensor> beta, c10::optional<Tensor> h, double eps, bool center) {
  check_f32(x, "x");
  TORCH_CHECK(x.dim() == 3, "x must be [T, S, W]");
  b200seq::StreamNormArgs p{};
  p.x = x.data_ptr<float>(); p.S = static_cast<int>(x.size(1)); p.W = static_cast<int>(x.size(2));
  const int64_t T = x.size(0);
  bool bf16 = false, have_dtype = false;
  auto act = [&](const Tensor& t, const char* name) {
    const bool is = act_is_bf16(t, name);
    TORCH_CHECK(!have_dtype || is == bf16, name, ": activation dtypes differ");
    bf16 = is; have_dtype = true;
  };
  auto vec = [&](const c10::optional<Tensor>& t, const char* name) -> const void* {
    if (!(t.has_value() && t->defined())) return nullptr;
    act(*t, name);
    TORCH_CHECK(t->is_contiguous() && t->numel() == p.W, name, " must hold W values");
    return t->data_ptr();
  };
  auto rows2 = [&](const c10::optional<Tensor>& t, const char* name, int64_t& ld) -> const void* {
    if (!(t.has_value() && t->defined())) return nullptr;
    act(*t, name);
    TORCH_CHECK(t->dim() == 2 && t->size(0) == T && t->size(1) == p.W && t->stride(1) == 1, name, " must be [T, W] with unit inner stride");
    ld = t->stride(0);
    return t->data_ptr();
  };
  p.a = rows2(a, "a", p.lda); p.b = rows2(b, "b", p.ldb);
  p.bias_a = vec(bias_a, "bias_a"); p.ls = vec(ls, "ls");
  p.scale_a = static_cast<float>(scale_a); p.scale_b = static_cast<float>(scale_b);
  if (p.a != nullptr) {
    TORCH_CHECK(mix.has_value() && outc.has_value(), "an update needs mix and out coefficients");
    check_f32(*mix, "mix"); check_f32(*outc, "outc");
    TORCH_CHECK(mix->numel() == p.S * p.S && outc->numel() == p.S, "mix must be [S, S], outc [S]");
    p.mix = mix->data_ptr<float>(); p.outc = outc->data_ptr<float>();
  }
  if (inp.has_value() && inp->defined()) {
    check_f32(*inp, "inp");
    TORCH_CHECK(inp->numel() == p.S && w.has_value() && h.has_value(), "inp must be [S]; the norm needs w and h");
    p.inp = inp->data_ptr<float>();
    p.w = vec(w, "w"); p.beta = vec(beta, "beta");
    act(*h, "h");
    TORCH_CHECK(h->is_contiguous() && h->numel() == T * p.W, "h must be contiguous [T, W]");
    p.h = h->data_ptr();
  }
  p.eps = static_cast<float>(eps); p.center = center ? 1 : 0;
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(b200seq::stream_mix_norm(p, static_cast<int>(T), bf16, cur_stream()), "stream_mix_norm: ", p.S, " streams of width ", p.W,
              " have no kernel instance");
  count(); check_last_error("stream_mix_norm");
}

void add_sinusoid(Tensor x, const Tensor& positions, const Tensor& freq) {
  check_f32(x, "x"); check_f32(freq, "freq");
  TORCH_CHECK(x.dim() == 2 && x.size(1) % 2 == 0 && freq.numel() == x.size(1) / 2, "x must be [T, W] with even W and W / 2 frequencies");
  TORCH_CHECK(positions.is_cuda() && positions.scalar_type() == at::kLong && positions.is_contiguous() && positions.numel() == x.size(0),
              "positions must be a contiguous int64 CUDA tensor [T]");
  c10::cuda::CUDAGuard g(x.device());
  b200seq::add_sinusoid(x.data_ptr<float>(), positions.data_ptr<int64_t>(), freq.data_ptr<float>(), static_cast<int>(x.size(0)),
                        static_cast<int>(x.size(1)), cur_stream());
  count(); check_last_error("add_sinusoid");
}

void head_rms_norm(const Tensor& x, const Tensor& w, Tensor y, double eps) {
  const bool bf16 = act_is_bf16(x, "x");
  check_rows(x, "x");
  TORCH_CHECK(w.scalar_type() == x.scalar_type() && w.is_contiguous() && w.numel() == x.size(2), "weight must hold one value per channel of a head");
  TORCH_CHECK(y.scalar_type() == x.scalar_type() && y.is_contiguous() && y.numel() == x.numel(), "bad y");
  c10::cuda::CUDAGuard g(x.device());
  b200seq::head_rms_norm(x.data_ptr(), x.stride(0), w.data_ptr(), y.data_ptr(), static_cast<int>(x.size(0)), static_cast<int>(x.size(1)),
                         static_cast<int>(x.size(2)), static_cast<float>(eps), bf16, cur_stream());
  count(); check_last_error("head_rms_norm");
}

void window_attention_paged(const Tensor& q, const Tensor& kcache, const Tensor& vcache, const Tensor& block_table, const Tensor& tok_req,
                            const Tensor& tok_len, c10::optional<Tensor> slopes, c10::optional<Tensor> gate, Tensor out, int64_t block_size,
                            double scale, int64_t window, bool sink, double out_scale, int64_t max_len, c10::optional<Tensor> dist_bias) {
  const bool bf16 = act_is_bf16(q, "q");
  check_rows(q, "q");
  TORCH_CHECK(kcache.scalar_type() == q.scalar_type() && vcache.scalar_type() == q.scalar_type() && kcache.dim() == 3 && vcache.dim() == 3 &&
              kcache.is_contiguous() && vcache.is_contiguous() && kcache.size(2) == q.size(2) && vcache.size(1) == kcache.size(1),
              "caches must be contiguous [slots, G, d] / [slots, G, dv] in q's dtype");
  check_i32(block_table, "block_table"); check_i32(tok_req, "tok_req"); check_i32(tok_len, "tok_len");
  b200seq::WindowAttnArgs p{};
  p.n_tok = static_cast<int>(q.size(0));
  p.H = static_cast<int>(q.size(1)); p.G = static_cast<int>(kcache.size(1)); p.d = static_cast<int>(q.size(2));
  p.dv = static_cast<int>(vcache.size(2));
  TORCH_CHECK(block_table.dim() == 2 && tok_req.numel() == q.size(0) && tok_len.numel() == q.size(0), "bad packed-batch tensors");
  TORCH_CHECK(out.scalar_type() == q.scalar_type() && out.is_contiguous() && out.numel() == q.size(0) * p.H * p.dv, "bad out");
  p.q = q.data_ptr(); p.ldq = q.stride(0); p.kcache = kcache.data_ptr(); p.vcache = vcache.data_ptr();
  p.block_table = block_table.data_ptr<int>(); p.tok_req = tok_req.data_ptr<int>(); p.tok_len = tok_len.data_ptr<int>();
  if (slopes.has_value() && slopes->defined()) {
    check_f32(*slopes, "slopes");
    TORCH_CHECK(slopes->numel() == p.H, "slopes must be [H]");
    p.slopes = slopes->data_ptr<float>();
  }
  if (dist_bias.has_value() && dist_bias->defined()) {
    check_f32(*dist_bias, "dist_bias");
    TORCH_CHECK(dist_bias->dim() == 2 && dist_bias->size(0) >= 1 && dist_bias->size(1) == p.H, "dist_bias must be [L, H]");
    p.dist_bias = dist_bias->data_ptr<float>(); p.n_bias = static_cast<int>(dist_bias->size(0));
  }
  if (gate.has_value() && gate->defined()) {
    check_act2(*gate, q, "gate");
    TORCH_CHECK(gate->size(0) == q.size(0) && gate->size(1) == p.H, "gate must be [T, H]");
    p.gate = gate->data_ptr(); p.ldg = gate->stride(0);
  }
  p.out = out.data_ptr();
  p.block_size = static_cast<int>(block_size); p.max_blocks = static_cast<int>(block_table.size(1));
  p.scale = static_cast<float>(scale); p.out_scale = static_cast<float>(out_scale);
  p.window = static_cast<int>(window); p.sink = sink ? 1 : 0;
  c10::cuda::CUDAGuard g(q.device());
  p.n_splits = 1;
  Tensor ws;
  if (block_table.size(0) == q.size(0) && q.size(0) > 0) {   // one token per sequence: a decoding batch
    p.decode = 1;
    const int64_t longest = max_len > 0 ? max_len : block_table.size(1) * block_size;      // unknown: what the tables can hold
    const int keys = static_cast<int>(window > 0 ? std::min<int64_t>(window, longest) : longest);
    p.n_splits = b200seq::window_attention_splits(p.H, p.G, p.n_tok, keys);
    if (p.n_splits > 1) {
      ws = torch::empty({q.size(0), p.H, p.n_splits, p.dv + 2}, q.options().dtype(at::kFloat));
      p.ws = ws.data_ptr<float>();
    }
  }
  TORCH_CHECK(b200seq::window_attention_paged(p, bf16, cur_stream()), "window_attention_paged: no kernel instance for heads ", p.H, " / ",
              p.G, ", dims ", p.d, " / ", p.dv);
  count(p.n_splits > 1 ? 2 : 1); check_last_error("window_attention_paged");
}

void sigmoid_attention_paged(const Tensor& q, const Tensor& kcache, const Tensor& vcache, const Tensor& block_table, const Tensor& tok_req,
                             const Tensor& tok_len, c10::optional<Tensor> head_bias, c10::optional<Tensor> turns_back, Tensor out,
                             int64_t block_size, double scale, double softcap, bool interleaved, int64_t max_len) {
  const bool bf16 = act_is_bf16(q, "q");
  check_rows(q, "q");
  TORCH_CHECK(kcache.scalar_type() == q.scalar_type() && vcache.scalar_type() == q.scalar_type() && kcache.dim() == 3 && vcache.dim() == 3 &&
              kcache.is_contiguous() && vcache.is_contiguous() && kcache.size(2) == q.size(2) && vcache.size(1) == kcache.size(1),
              "caches must be contiguous [slots, G, d] / [slots, G, dv] in q's dtype");
  check_i32(block_table, "block_table"); check_i32(tok_req, "tok_req"); check_i32(tok_len, "tok_len");
  b200seq::WindowAttnArgs p{};
  p.n_tok = static_cast<int>(q.size(0));
  p.H = static_cast<int>(q.size(1)); p.G = static_cast<int>(kcache.size(1)); p.d = static_cast<int>(q.size(2));
  p.dv = static_cast<int>(vcache.size(2));
  TORCH_CHECK(block_table.dim() == 2 && tok_req.numel() == q.size(0) && tok_len.numel() == q.size(0), "bad packed-batch tensors");
  TORCH_CHECK(out.scalar_type() == q.scalar_type() && out.is_contiguous() && out.numel() == q.size(0) * p.H * p.dv, "bad out");
  p.q = q.data_ptr(); p.ldq = q.stride(0); p.kcache = kcache.data_ptr(); p.vcache = vcache.data_ptr();
  p.block_table = block_table.data_ptr<int>(); p.tok_req = tok_req.data_ptr<int>(); p.tok_len = tok_len.data_ptr<int>();
  if (opt_ptr(head_bias) != nullptr) {
    check_f32(*head_bias, "head_bias");
    TORCH_CHECK(head_bias->numel() == p.H, "head_bias must be [H]");
    p.slopes = head_bias->data_ptr<float>();
  }
  if (opt_ptr(turns_back) != nullptr) {
    check_f32(*turns_back, "turns_back");
    TORCH_CHECK(turns_back->dim() == 2 && turns_back->size(1) == 2 && 2 * turns_back->size(0) <= p.dv, "turns_back must be [n, 2], 2 n <= dv");
    p.turns_back = turns_back->data_ptr<float>(); p.n_turn = static_cast<int>(turns_back->size(0)); p.interleaved = interleaved ? 1 : 0;
  }
  p.out = out.data_ptr();
  p.block_size = static_cast<int>(block_size); p.max_blocks = static_cast<int>(block_table.size(1));
  p.scale = static_cast<float>(scale); p.out_scale = 1.f; p.softcap = static_cast<float>(softcap);
  c10::cuda::CUDAGuard g(q.device());
  p.n_splits = 1;
  Tensor ws;
  if (block_table.size(0) == q.size(0) && q.size(0) > 0) {   // one token per sequence: a decoding batch
    p.decode = 1;
    const int64_t longest = max_len > 0 ? max_len : block_table.size(1) * block_size;      // unknown: what the tables can hold
    p.n_splits = b200seq::window_attention_splits(p.H, p.G, p.n_tok, static_cast<int>(longest));
    if (p.n_splits > 1) {
      ws = torch::empty({q.size(0), p.H, p.n_splits, p.dv + 2}, q.options().dtype(at::kFloat));
      p.ws = ws.data_ptr<float>();
    }
  }
  TORCH_CHECK(b200seq::sigmoid_attention_paged(p, bf16, cur_stream()), "sigmoid_attention_paged: no kernel instance for heads ", p.H, " / ", p.G,
              ", dims ", p.d, " / ", p.dv);
  count(p.n_splits > 1 ? 2 : 1); check_last_error("sigmoid_attention_paged");
}

void gated_add_norm(Tensor x, c10::optional<Tensor> a, c10::optional<Tensor> ga, c10::optional<Tensor> bias_a, c10::optional<Tensor> b,
                    c10::optional<Tensor> gb, c10::optional<Tensor> bias_b, const Tensor& w1, c10::optional<Tensor> w2, Tensor h1,
                    c10::optional<Tensor> h2, double eps, bool center) {
  check_f32(x, "x");
  const bool bf16 = act_is_bf16(h1, "h1");
  TORCH_CHECK(x.dim() == 2 && h1.is_contiguous() && h1.sizes() == x.sizes(), "x / h1 must be [rows, cols]");
  b200seq::GatedNormArgs p{};
  p.x = x.data_ptr<float>(); p.W = static_cast<int>(x.size(1)); p.center = center ? 1 : 0; p.eps = static_cast<float>(eps);
  auto rows = [&](const c10::optional<Tensor>& t, const char* name, const void** ptr, int64_t* ld) {
    if (opt_ptr(t) == nullptr) return;
    check_act2(*t, h1, name);
    TORCH_CHECK(t->sizes() == x.sizes(), name, " must be shaped like x");
    *ptr = t->data_ptr(); *ld = t->stride(0);
  };
  auto vec = [&](const Tensor& t, const char* name) -> const void* {
    TORCH_CHECK(t.is_cuda() && t.scalar_type() == h1.scalar_type() && t.is_contiguous() && t.numel() == x.size(1), name,
                " must be a contiguous [cols] tensor in h1's dtype");
    return t.data_ptr();
  };
  rows(a, "a", &p.a, &p.lda); rows(ga, "gate_a", &p.ga, &p.ldga); rows(b, "b", &p.b, &p.ldb); rows(gb, "gate_b", &p.gb, &p.ldgb);
  TORCH_CHECK((p.ga == nullptr || p.a != nullptr) && (p.gb == nullptr || p.b != nullptr), "a gate without an addend");
  if (opt_ptr(bias_a) != nullptr) p.bias_a = vec(*bias_a, "bias_a");
  if (opt_ptr(bias_b) != nullptr) p.bias_b = vec(*bias_b, "bias_b");
  p.w1 = vec(w1, "weight1"); p.h1 = h1.data_ptr();
  if (opt_ptr(h2) != nullptr) {
    TORCH_CHECK(opt_ptr(w2) != nullptr && h2->is_contiguous() && h2->sizes() == x.sizes() && h2->scalar_type() == h1.scalar_type(), "bad h2");
    p.w2 = vec(*w2, "weight2"); p.h2 = h2->data_ptr();
  }
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(b200seq::gated_add_norm(p, static_cast<int>(x.size(0)), bf16, cur_stream()), "gated_add_norm: rows of ", p.W, " are too wide");
  count(); check_last_error("gated_add_norm");
}

void squash_add(Tensor x, c10::optional<Tensor> a, c10::optional<Tensor> alpha_o, c10::optional<Tensor> wo, c10::optional<Tensor> bo,
                c10::optional<Tensor> alpha_n, c10::optional<Tensor> wn, c10::optional<Tensor> bn, c10::optional<Tensor> h, double mult,
                double x_scale) {
  check_f32(x, "x");
  TORCH_CHECK(x.dim() == 2, "x must be [rows, cols]");
  b200seq::SquashArgs p{};
  p.x = x.data_ptr<float>(); p.W = static_cast<int>(x.size(1)); p.mult = static_cast<float>(mult); p.x_scale = static_cast<float>(x_scale);
  const Tensor* like = opt_ptr(h) != nullptr ? &*h : (opt_ptr(a) != nullptr ? &*a : nullptr);
  const bool bf16 = like != nullptr && act_is_bf16(*like, "h");
  auto vec = [&](const c10::optional<Tensor>& t, int64_t n, const char* name) -> const void* {
    TORCH_CHECK(opt_ptr(t) != nullptr && t->is_cuda() && t->scalar_type() == like->scalar_type() && t->is_contiguous() && t->numel() == n, name,
                " must be a contiguous tensor of ", n, " in the activations' dtype");
    return t->data_ptr();
  };
  if (opt_ptr(a) != nullptr) {
    check_act2(*a, *like, "a");
    TORCH_CHECK(a->sizes() == x.sizes(), "a must be shaped like x");
    p.a = a->data_ptr(); p.lda = a->stride(0);
    if (opt_ptr(wo) != nullptr) { p.wo = vec(wo, p.W, "weight"); p.bo = vec(bo, p.W, "bias"); p.alpha_o = vec(alpha_o, 1, "alpha"); }
  }
  if (opt_ptr(h) != nullptr) {
    TORCH_CHECK(h->is_contiguous() && h->sizes() == x.sizes(), "h must be contiguous and shaped like x");
    p.h = h->data_ptr(); p.wn = vec(wn, p.W, "next weight"); p.bn = vec(bn, p.W, "next bias"); p.alpha_n = vec(alpha_n, 1, "next alpha");
  }
  c10::cuda::CUDAGuard g(x.device());
  b200seq::squash_add(p, static_cast<int>(x.size(0)), bf16, cur_stream());
  count(); check_last_error("squash_add");
}

void head_rotary(const std::vector<Tensor>& x, const std::vector<c10::optional<Tensor>>& turns, const std::vector<c10::optional<Tensor>>& weight,
                 const std::vector<c10::optional<Tensor>>& out, const std::vector<c10::optional<Tensor>>& pages,
                 const std::vector<bool>& interleaved, const std::vector<double>& amplitude, const std::vector<bool>& back,
                 const std::vector<bool>& rms, const std::vector<int64_t>& out_half, const std::vector<c10::optional<Tensor>>& table,
                 const Tensor& positions, c10::optional<Tensor> slots, double eps) {
  const size_t n = x.size();
  TORCH_CHECK(n >= 1 && n <= 3 && turns.size() == n && weight.size() == n && out.size() == n && pages.size() == n && interleaved.size() == n &&
              amplitude.size() == n && back.size() == n && rms.size() == n && out_half.size() == n && table.size() == n, "one to three parts");
  const bool bf16 = act_is_bf16(x[0], "x");
  const int64_t T = x[0].size(0);
  TORCH_CHECK(positions.is_cuda() && positions.scalar_type() == at::kLong && positions.is_contiguous() && positions.numel() == T,
              "positions must be int64 [T]");
  b200seq::HeadRotaryArgs p{};
  p.n_parts = static_cast<int>(n); p.eps = static_cast<float>(eps); p.positions = positions.data_ptr<int64_t>();
  if (opt_ptr(slots) != nullptr) {
    TORCH_CHECK(slots->is_cuda() && slots->scalar_type() == at::kLong && slots->is_contiguous() && slots->numel() == T, "slots must be int64 [T]");
    p.slots = slots->data_ptr<int64_t>();
  }
  for (size_t k = 0; k < n; ++k) {
    b200seq::RotPart& r = p.part[k];
    TORCH_CHECK(x[k].is_cuda() && x[k].dim() == 3 && x[k].size(0) == T && x[k].stride(2) == 1 && x[k].scalar_type() == x[0].scalar_type(),
                "x must be [T, heads, d] with unit inner stride, all of one dtype");
    r.x = x[k].data_ptr(); r.ld_x = x[k].stride(0); r.hs_x = x[k].stride(1);
    r.heads = static_cast<int>(x[k].size(1)); r.d = static_cast<int>(x[k].size(2));
    r.interleaved = interleaved[k]; r.back = back[k]; r.rms = rms[k]; r.amplitude = static_cast<float>(amplitude[k]);
    if (opt_ptr(turns[k]) != nullptr) {
      check_f32(*turns[k], "turns");
      TORCH_CHECK(turns[k]->dim() == 2 && turns[k]->size(1) == 2 && 2 * turns[k]->size(0) <= r.d, "turns must be [n, 2] with 2 n <= d");
      r.turns = turns[k]->data_ptr<float>(); r.n_turn = static_cast<int>(turns[k]->size(0));
    }
    if (opt_ptr(table[k]) != nullptr) {
      check_f32(*table[k], "table");
      TORCH_CHECK(table[k]->numel() == T * r.n_turn * 2, "table must be [T, n, 2]");
      r.table = table[k]->data_ptr<float>();
    }
    if (opt_ptr(weight[k]) != nullptr) {
      TORCH_CHECK(weight[k]->scalar_type() == x[0].scalar_type() && weight[k]->is_contiguous() && weight[k]->numel() == r.d, "bad weight");
      r.weight = weight[k]->data_ptr();
    }
    auto dst = [&](const Tensor& t, const char* name) {
      TORCH_CHECK(t.is_cuda() && t.dim() == 3 && t.stride(2) == 1 && t.size(1) == r.heads && t.size(2) >= r.d && t.scalar_type() == x[0].scalar_type(),
                  name, " must be [., heads, d] with unit inner stride in x's dtype");
    };
    if (opt_ptr(out[k]) != nullptr) {
      dst(*out[k], "out");
      TORCH_CHECK(out[k]->size(0) == T, "out must have one row per token");
      r.out = out[k]->data_ptr(); r.ld_out = out[k]->stride(0); r.hs_out = out[k]->stride(1); r.d_out = static_cast<int>(out[k]->size(2));
      r.out_half = static_cast<int>(out_half[k]);
      TORCH_CHECK(r.out_half == 0 || (r.out_half >= r.d / 2 && r.out_half + r.d - r.d / 2 <= r.d_out), "bad out_half");
    }
    if (opt_ptr(pages[k]) != nullptr) {
      dst(*pages[k], "pages");
      TORCH_CHECK(p.slots != nullptr, "pages need slots");
      r.pages = pages[k]->data_ptr(); r.ld_page = pages[k]->stride(0); r.hs_page = pages[k]->stride(1);
    }
  }
  c10::cuda::CUDAGuard g(x[0].device());
  TORCH_CHECK(b200seq::head_rotary(p, static_cast<int>(T), bf16, cur_stream()), "head_rotary: heads too wide");
  count(); check_last_error("head_rotary");
}

void latent_head_assemble(const Tensor& q, const Tensor& k, const Tensor& k_rot, const Tensor& v, c10::optional<Tensor> turns, bool interleaved,
                          double amplitude, const Tensor& positions, Tensor q_out, Tensor k_out, Tensor v_out) {
  const bool bf16 = act_is_bf16(q, "q");
  const auto dt = q.scalar_type();
  TORCH_CHECK(q.dim() == 3 && k.dim() == 3 && v.dim() == 3 && q.stride(2) == 1 && q.stride(1) == q.size(2) && k.is_contiguous() && v.is_contiguous() &&
              k.scalar_type() == dt && v.scalar_type() == dt, "q / k / v must be [T, H, .] of one dtype, k and v contiguous, q with contiguous heads");
  check_act2(k_rot, q, "k_rot");
  b200seq::LatentHeadArgs p{};
  const int64_t T = q.size(0);
  p.H = static_cast<int>(q.size(1)); p.d = static_cast<int>(k.size(2)); p.n = static_cast<int>(k_rot.size(1)); p.dv = static_cast<int>(v.size(2));
  TORCH_CHECK(q.size(2) == p.d + p.n && k.size(0) == T && v.size(0) == T && k.size(1) == p.H && v.size(1) == p.H && k_rot.size(0) == T, "bad shapes");
  TORCH_CHECK(positions.is_cuda() && positions.scalar_type() == at::kLong && positions.is_contiguous() && positions.numel() == T, "bad positions");
  p.width = static_cast<int>(q_out.size(2));
  for (const Tensor* o : {&q_out, &k_out, &v_out})
    TORCH_CHECK(o->is_contiguous() && o->scalar_type() == dt && o->dim() == 3 && o->size(0) == T && o->size(1) == p.H && o->size(2) == p.width, "bad outputs");
  TORCH_CHECK(p.width >= p.d + p.n && p.width >= p.dv, "outputs too narrow");
  if (opt_ptr(turns) != nullptr) {
    check_f32(*turns, "turns");
    TORCH_CHECK(turns->dim() == 2 && turns->size(1) == 2 && 2 * turns->size(0) <= p.n, "turns must be [pairs, 2]");
    p.turns = turns->data_ptr<float>(); p.n_turn = static_cast<int>(turns->size(0));
  }
  p.q = q.data_ptr(); p.ld_q = q.stride(0); p.k = k.data_ptr(); p.k_rot = k_rot.data_ptr(); p.ld_kr = k_rot.stride(0); p.v = v.data_ptr();
  p.positions = positions.data_ptr<int64_t>(); p.q_out = q_out.data_ptr(); p.k_out = k_out.data_ptr(); p.v_out = v_out.data_ptr();
  p.interleaved = interleaved ? 1 : 0; p.amplitude = static_cast<float>(amplitude);
  c10::cuda::CUDAGuard g(q.device());
  TORCH_CHECK(b200seq::latent_head_assemble(p, static_cast<int>(T), bf16, cur_stream()), "latent_head_assemble: too many pairs");
  count(); check_last_error("latent_head_assemble");
}

void head_gate(const Tensor& o, const Tensor& gate, Tensor y) {
  const bool bf16 = act_is_bf16(y, "y");
  TORCH_CHECK(o.is_cuda() && o.dim() == 3 && o.stride(2) == 1 && y.is_contiguous() && y.sizes() == o.sizes() &&
              (o.scalar_type() == y.scalar_type() || o.scalar_type() == at::kFloat), "o must be [T, H, dv], fp32 or in y's dtype");
  check_act2(gate, y, "gate");
  const bool per_element = gate.size(1) == o.size(1) * o.size(2);
  TORCH_CHECK(gate.size(0) == o.size(0) && (per_element || gate.size(1) == o.size(1)), "gate must be [T, H] or [T, H * dv]");
  c10::cuda::CUDAGuard g(o.device());
  b200seq::head_gate(o.data_ptr(), o.scalar_type() == at::kFloat, o.stride(0), o.stride(1), gate.data_ptr(), gate.stride(0), per_element,
                     y.data_ptr(), static_cast<int>(o.size(0)), static_cast<int>(o.size(1)), static_cast<int>(o.size(2)), bf16, cur_stream());
  count(); check_last_error("head_gate");
}

void rglru_scan(const Tensor& u, const Tensor& w, const Tensor& bias, const Tensor& lam, c10::optional<Tensor> y_pre, const Tensor& cu,
                const Tensor& rows, Tensor state, Tensor y, double decay_scale, int64_t max_len) {
  const bool bf16 = act_is_bf16(u, "u");
  check_act2(u, u, "u"); check_f32(state, "state"); check_i32(cu, "cu"); check_i32(rows, "rows");
  b200seq::LruArgs p{};
  p.n_tok = static_cast<int>(u.size(0)); p.C = static_cast<int>(u.size(1));
  TORCH_CHECK(w.scalar_type() == u.scalar_type() && w.is_contiguous() && w.dim() == 4 && w.size(1) == 2 && w.size(2) == w.size(3) &&
              w.size(0) * w.size(2) == p.C, "gate weights must be contiguous [B, 2, n, n] with B n channels");
  p.n_blocks = static_cast<int>(w.size(0)); p.n = static_cast<int>(w.size(2));
  TORCH_CHECK(bias.scalar_type() == u.scalar_type() && bias.is_contiguous() && bias.numel() == 2 * p.C && lam.scalar_type() == u.scalar_type() &&
              lam.is_contiguous() && lam.numel() == p.C, "bad gate bias / lam");
  TORCH_CHECK(state.dim() == 2 && state.size(1) == p.C && y.is_contiguous() && y.sizes() == u.sizes() && y.scalar_type() == u.scalar_type(), "bad state / y");
  if (opt_ptr(y_pre) != nullptr) {
    check_act2(*y_pre, u, "y_pre");
    TORCH_CHECK(y_pre->sizes() == u.sizes(), "bad y_pre");
    p.y_pre = y_pre->data_ptr(); p.ldy = y_pre->stride(0);
  }
  p.u = u.data_ptr(); p.ldu = u.stride(0); p.w = w.data_ptr(); p.bias = bias.data_ptr(); p.lam = lam.data_ptr();
  p.cu = cu.data_ptr<int>(); p.rows = rows.data_ptr<int>(); p.state = state.data_ptr<float>(); p.y = y.data_ptr();
  p.decay_scale = static_cast<float>(decay_scale);
  const int R = static_cast<int>(rows.numel());
  c10::cuda::CUDAGuard g(u.device());
const int longest = static_cast<int>(max_len > 0 ? max_len : p.n_tok);
  auto workspace = [&]() {
    Tensor ws = torch::empty({R, p.max_runs, u.size(1), 2}, state.options());
    p.ws = ws.data_ptr<float>();
    return ws;
  };
  if (longest == 1) {
    TORCH_CHECK(b200seq::rglru_step(p, R, bf16, cur_stream()), "rglru_scan: unsupported sizes");
    count();
  } else if (bf16 && b200seq::rglru_chunked_supported(p, longest)) {
    p.max_runs = b200seq::lru_chunks(longest);
    Tensor ws = workspace();
    TORCH_CHECK(b200seq::rglru_scan_chunked(p, R, cur_stream()), "rglru_scan: the chunked kernel could not be launched");
    count(3);
  } else {
    p.max_runs = b200seq::lru_runs(longest);
    Tensor pre = torch::empty({u.size(0), 2, u.size(1)}, state.options()), ws;
    p.pre = pre.data_ptr<float>();
    if (p.max_runs > 1) ws = workspace();
    TORCH_CHECK(b200seq::rglru_scan(p, R, bf16, cur_stream()), "rglru_scan: too many gate blocks (", p.n_blocks, ")");
    count(p.max_runs > 1 ? 4 : 2);
  }
  check_last_error("rglru_scan");
}

void selective_scan(const Tensor& x, c10::optional<Tensor> z, const Tensor& B, const Tensor& Cm, const Tensor& dt_pre,
                    c10::optional<Tensor> dt_bias, const Tensor& A_log, const Tensor& D, const Tensor& cu, const Tensor& rows, Tensor state,
                    Tensor y, double out_scale) {
  const bool bf16 = act_is_bf16(x, "x");
  check_act2(x, x, "x"); check_act2(B, x, "B"); check_act2(Cm, x, "C"); check_act2(y, x, "y");
  check_f32(state, "state"); check_i32(cu, "cu"); check_i32(rows, "rows");
  b200seq::SelScanArgs p{};
  p.C = static_cast<int>(x.size(1)); p.N = static_cast<int>(B.size(1));
  const int64_t T = x.size(0);
  TORCH_CHECK(B.size(0) == T && Cm.size(0) == T && Cm.size(1) == p.N && y.size(0) == T && y.size(1) == p.C, "bad B / C / y shapes");
  TORCH_CHECK(dt_pre.is_cuda() && dt_pre.scalar_type() == at::kFloat && dt_pre.dim() == 2 && dt_pre.stride(1) == 1 && dt_pre.size(0) == T &&
              dt_pre.size(1) == p.C, "dt_pre must be fp32 [T, C]");
  TORCH_CHECK(state.dim() == 3 && state.size(1) == p.C && state.size(2) == p.N, "state must be [rows, C, N]");
  TORCH_CHECK(A_log.scalar_type() == x.scalar_type() && A_log.is_contiguous() && A_log.numel() == static_cast<int64_t>(p.C) * p.N &&
              D.scalar_type() == x.scalar_type() && D.is_contiguous() && D.numel() == p.C, "bad A_log / D");
  if (z.has_value() && z->defined()) { check_act2(*z, x, "z"); TORCH_CHECK(z->size(0) == T && z->size(1) == p.C, "bad z"); p.z = z->data_ptr(); p.ldz = z->stride(0); }
  if (dt_bias.has_value() && dt_bias->defined()) {
    TORCH_CHECK(dt_bias->scalar_type() == x.scalar_type() && dt_bias->is_contiguous() && dt_bias->numel() == p.C, "bad dt_bias");
    p.dt_bias = dt_bias->data_ptr();
  }
  p.x = x.data_ptr(); p.B = B.data_ptr(); p.Cm = Cm.data_ptr(); p.y = y.data_ptr(); p.dt_pre = dt_pre.data_ptr<float>();
  p.ldx = x.stride(0); p.ldb = B.stride(0); p.ldc = Cm.stride(0); p.ldy = y.stride(0); p.lddt = dt_pre.stride(0);
  p.A_log = A_log.data_ptr(); p.D = D.data_ptr();
  p.cu = cu.data_ptr<int>(); p.rows = rows.data_ptr<int>(); p.state = state.data_ptr<float>();
  p.out_scale = static_cast<float>(out_scale);
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(b200seq::selective_scan(p, static_cast<int>(rows.numel()), bf16, cur_stream()), "selective_scan: ", p.N,
              " states per channel exceed the largest kernel instance (128)");
  count(); check_last_error("selective_scan");
}
}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.def("add_rms_norm", &add_rms_norm);
  m.def("retention_scan", &retention_scan);
  m.def("poly_norm", &poly_norm);
  m.def("gelu_mul", &gelu_mul);
  m.def("decay_gates", &decay_gates);
  m.def("gated_head_rms_norm", &gated_head_rms_norm);
  m.def("causal_conv", &causal_conv);
  m.def("stream_mix_norm", &stream_mix_norm);
  m.def("add_sinusoid", &add_sinusoid);
  m.def("head_rms_norm", &head_rms_norm);
  m.def("window_attention_paged", &window_attention_paged);
  m.def("selective_scan", &selective_scan);
  m.def("sigmoid_attention_paged", &sigmoid_attention_paged);
  m.def("gated_add_norm", &gated_add_norm);
  m.def("head_rotary", &head_rotary);
  m.def("squash_add", &squash_add);
  m.def("latent_head_assemble", &latent_head_assemble);
  m.def("head_gate", &head_gate);
  m.def("rglru_scan", &rglru_scan);
  m.def("rglru_status", []() { return b200seq::rglru_chunked_status(); });
  m.def("delta_rule_scan", &delta_rule_scan);
  m.def("mlstm_scan", &mlstm_scan);
  m.def("latent_attention_paged", &latent_attention_paged);
  m.def("group_limited_router", &group_limited_router);
  m.def("norm_add", &norm_add);
  m.def("norm_rope", &norm_rope);
  m.def("mixed_attention_paged", &mixed_attention_paged);
  m.def("gen_delta_scan", &gen_delta_scan);
  m.def("mingru_scan", &mingru_scan);
  m.def("clamped_glu", &clamped_glu);
  m.def("launch_count", []() { return g_launches.load(); });
  m.def("reset_launch_count", []() { g_launches.store(0); });
}
