// Bindings of the attention / decode / sampling / fused-loss launchers.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include "api.h"

namespace {
// Also clears this thread's "last error" slot: launchers report cudaGetLastError() after their
// launch, and an unrelated, already handled status left there by another library (for example
// cudaErrorNotReady from an event query) must not be mistaken for a launch failure.
inline cudaStream_t cur_stream() {
  (void)cudaGetLastError();
  return at::cuda::getCurrentCUDAStream().stream();
}
inline void check(int rc, const char* what) {
  if (rc != 0) {
    char buf[160];
    snprintf(buf, sizeof(buf), "%s failed with code %d (%s)", what, rc, rc > 0 ? cudaGetErrorString((cudaError_t)rc) : "argument check");
    fprintf(stderr, "[relax_b200] %s\n", buf);
    throw std::runtime_error(buf);
  }
}

void fa_bwd(torch::Tensor q, torch::Tensor k, torch::Tensor v, torch::Tensor o, torch::Tensor d_o, torch::Tensor lse,
            torch::Tensor dq, torch::Tensor dk, torch::Tensor dv, torch::Tensor delta, torch::Tensor dq_acc,
            torch::Tensor cu_q, torch::Tensor cu_k, int64_t max_kv_blocks, bool causal, double scale, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(q.device());
  check(rb_fa_bwd(q.data_ptr(), k.data_ptr(), v.data_ptr(), o.data_ptr(), d_o.data_ptr(), lse.data_ptr<float>(),
                  dq.data_ptr(), dk.data_ptr(), dv.data_ptr(), delta.data_ptr<float>(), dq_acc.data_ptr<float>(),
                  cu_q.data_ptr<int>(), cu_k.data_ptr<int>(), (int)cu_q.numel() - 1, (int)q.size(0), (int)k.size(0),
                  (int)q.size(1), (int)k.size(1), causal, (float)scale, (int)max_kv_blocks, err.data_ptr<int>(),
                  cur_stream()),
        "rb_fa_bwd");
}
int64_t decode_attn_splits(int64_t B, int64_t Hkv, int64_t max_ctx) {
  return rb_decode_attn_splits((int)B, (int)Hkv, (int)max_ctx);
}
void decode_attn(torch::Tensor q, torch::Tensor kc, torch::Tensor vc, torch::Tensor block_tables, torch::Tensor ctx_lens,
                 torch::Tensor out, c10::optional<torch::Tensor> part_o, c10::optional<torch::Tensor> part_ml,
                 int64_t max_ctx, double scale, int64_t splits, int64_t version, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(q.device());
  TORCH_CHECK(q.scalar_type() == at::kBFloat16 && q.size(2) == 128, "decode attention: bf16, head_dim 128");
  if (version == 3) {
    check(rb_decode_attn_tc(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), block_tables.data_ptr<int>(), ctx_lens.data_ptr<int>(),
                            out.data_ptr(), part_o.has_value() ? part_o->data_ptr<float>() : nullptr,
                            part_ml.has_value() ? part_ml->data_ptr<float>() : nullptr, (int)q.size(0), (int)q.size(1),
                            (int)kc.size(2), (int)kc.size(0), (int)kc.size(1), (int)block_tables.size(1), (int)max_ctx,
                            (float)scale, (int)splits, err.data_ptr<int>(), cur_stream()),
          "rb_decode_attn_tc");
    return;
  }
  auto fn = version == 1 ? rb_decode_attn_v1 : rb_decode_attn;
  check(fn(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), block_tables.data_ptr<int>(), ctx_lens.data_ptr<int>(),
                       out.data_ptr(), part_o.has_value() ? part_o->data_ptr<float>() : nullptr,
                       part_ml.has_value() ? part_ml->data_ptr<float>() : nullptr, (int)q.size(0), (int)q.size(1),
                       (int)kc.size(2), (int)kc.size(1), (int)block_tables.size(1), (int)max_ctx, (float)scale,
                       (int)splits, cur_stream()),
        "rb_decode_attn");
}
void sample(torch::Tensor logits, torch::Tensor temperature, torch::Tensor top_k, torch::Tensor top_p,
            torch::Tensor uniform, torch::Tensor tok, torch::Tensor logp, int64_t V) {
  const c10::cuda::CUDAGuard guard(logits.device());
  check(rb_sample(logits.data_ptr<float>(), (int)logits.size(0), (int)V, (int)logits.stride(0),
                  temperature.data_ptr<float>(), (const long long*)top_k.data_ptr<int64_t>(), top_p.data_ptr<float>(),
                  uniform.data_ptr<float>(), (long long*)tok.data_ptr<int64_t>(), logp.data_ptr<float>(), cur_stream()),
        "rb_sample");
}
void policy_loss(torch::Tensor ppo_kl, torch::Tensor adv, torch::Tensor loss, torch::Tensor clipfrac, torch::Tensor dkl,
                 double eps_clip, double eps_clip_high, double eps_clip_c) {
  const c10::cuda::CUDAGuard guard(ppo_kl.device());
  TORCH_CHECK(ppo_kl.scalar_type() == at::kFloat && adv.scalar_type() == at::kFloat, "fp32 inputs");
  TORCH_CHECK(ppo_kl.is_contiguous() && adv.is_contiguous() && adv.numel() == ppo_kl.numel(), "contiguous inputs of one size");
  check(rb_policy_loss(ppo_kl.data_ptr<float>(), adv.data_ptr<float>(), loss.data_ptr<float>(), clipfrac.data_ptr<float>(),
                       dkl.data_ptr<float>(), ppo_kl.numel(), (float)eps_clip, (float)eps_clip_high, (float)eps_clip_c,
                       cur_stream()),
        "rb_policy_loss");
}
void grouped_gemm_fwd(torch::Tensor X, torch::Tensor W, torch::Tensor Y, torch::Tensor tile_expert, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(X.device());
  TORCH_CHECK(X.scalar_type() == at::kBFloat16 && W.scalar_type() == at::kBFloat16 && Y.scalar_type() == at::kBFloat16, "bf16 only");
  TORCH_CHECK(X.is_contiguous() && W.is_contiguous() && Y.is_contiguous() && W.dim() == 3, "contiguous X [cap,K], W [E,N,K]");
  TORCH_CHECK(tile_expert.scalar_type() == at::kInt && tile_expert.numel() * 128 == X.size(0), "tile map: one int32 per 128 rows");
  check(rb_grouped_gemm_fwd(X.data_ptr(), W.data_ptr(), Y.data_ptr(), tile_expert.data_ptr<int>(), (int)X.size(0),
                            (int)W.size(1), (int)W.size(2), (int)W.size(0), err.data_ptr<int>(), cur_stream()),
        "rb_grouped_gemm_fwd");
}
void grouped_gemm_dgrad(torch::Tensor dY, torch::Tensor W, torch::Tensor dX, torch::Tensor tile_expert, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(dY.device());
  TORCH_CHECK(dY.scalar_type() == at::kBFloat16 && W.scalar_type() == at::kBFloat16 && dX.scalar_type() == at::kBFloat16, "bf16 only");
  TORCH_CHECK(dY.is_contiguous() && W.is_contiguous() && dX.is_contiguous() && W.dim() == 3, "contiguous dY [cap,N], W [E,N,K]");
  TORCH_CHECK(tile_expert.scalar_type() == at::kInt && tile_expert.numel() * 128 == dY.size(0), "tile map: one int32 per 128 rows");
  check(rb_grouped_gemm_dgrad(dY.data_ptr(), W.data_ptr(), dX.data_ptr(), tile_expert.data_ptr<int>(), (int)dY.size(0),
                              (int)W.size(1), (int)W.size(2), (int)W.size(0), err.data_ptr<int>(), cur_stream()),
        "rb_grouped_gemm_dgrad");
}
void grouped_gemm_wgrad(torch::Tensor dY, torch::Tensor X, torch::Tensor dW, torch::Tensor expert_rows, bool accumulate,
                        torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(dY.device());
  TORCH_CHECK(dY.scalar_type() == at::kBFloat16 && X.scalar_type() == at::kBFloat16, "bf16 inputs");
  TORCH_CHECK(dY.is_contiguous() && X.is_contiguous() && dW.is_contiguous() && dW.dim() == 3, "contiguous dY, X, dW [E,N,K]");
  TORCH_CHECK(expert_rows.scalar_type() == at::kInt && expert_rows.numel() == dW.size(0) + 1, "expert_rows: int32 [E + 1]");
  const bool f32 = dW.scalar_type() == at::kFloat;
  TORCH_CHECK(f32 || dW.scalar_type() == at::kBFloat16, "dW must be fp32 or bf16");
  check(rb_grouped_gemm_wgrad(dY.data_ptr(), X.data_ptr(), dW.data_ptr(), expert_rows.data_ptr<int>(), (int)dY.size(0),
                              (int)dW.size(1), (int)dW.size(2), (int)dW.size(0), f32, accumulate, err.data_ptr<int>(),
                              cur_stream()),
        "rb_grouped_gemm_wgrad");
}
void topk_router(torch::Tensor logits, int64_t K, bool norm, torch::Tensor w, torch::Tensor idx, torch::Tensor probs) {
  const c10::cuda::CUDAGuard guard(logits.device());
  check(rb_topk_router(logits.data_ptr<float>(), (int)logits.size(0), (int)logits.size(1), (int)K, norm,
                       w.data_ptr<float>(), (long long*)idx.data_ptr<int64_t>(), probs.data_ptr<float>(), cur_stream()),
        "rb_topk_router");
}
int64_t lm_head_splits(int64_t M, int64_t N) { return rb_lm_head_splits((int)M, (int)N); }
void lm_head_logprob(torch::Tensor h, torch::Tensor W, torch::Tensor targets, torch::Tensor partials, int64_t vocab_start,
                     double inv_temp, int64_t n_splits, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(h.device());
  TORCH_CHECK(h.scalar_type() == at::kBFloat16 && W.scalar_type() == at::kBFloat16, "fused LM head: bf16");
  check(rb_lm_head_logprob(h.data_ptr(), W.data_ptr(), (const long long*)targets.data_ptr<int64_t>(),
                           partials.data_ptr<float>(), (int)h.size(0), (int)W.size(0), (int)h.size(1), (int)h.stride(0),
                           (int)W.stride(0), (int)vocab_start, (float)inv_temp, (int)n_splits, err.data_ptr<int>(),
                           cur_stream()),
        "rb_lm_head_logprob");
}
void lm_head_dlogits(torch::Tensor h, torch::Tensor W, torch::Tensor targets, torch::Tensor row_stats, torch::Tensor g_lp,
                     c10::optional<torch::Tensor> g_ent, torch::Tensor dlogits, int64_t vocab_start, double inv_temp,
                     torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(h.device());
  check(rb_lm_head_dlogits(h.data_ptr(), W.data_ptr(), (const long long*)targets.data_ptr<int64_t>(),
                           row_stats.data_ptr<float>(), g_lp.data_ptr<float>(),
                           g_ent.has_value() ? g_ent->data_ptr<float>() : nullptr, dlogits.data_ptr(), (int)h.size(0),
                           (int)W.size(0), (int)h.size(1), (int)h.stride(0), (int)W.stride(0), (int)dlogits.stride(0),
                           (int)vocab_start, (float)inv_temp, err.data_ptr<int>(), cur_stream()),
        "rb_lm_head_dlogits");
}
}  // namespace

void register_symm(pybind11::module_& m);
void register_fused(pybind11::module_& m);
void register_vmm(pybind11::module_& m);

void register_more(pybind11::module_& m) {
  register_symm(m);
  register_fused(m);
  register_vmm(m);
  m.def("fa_bwd", &fa_bwd);
  m.def("decode_attn_splits", &decode_attn_splits);
  m.def("decode_attn", &decode_attn);
  m.def("sample", &sample);
  m.def("policy_loss", &policy_loss);
  m.def("grouped_gemm_fwd", &grouped_gemm_fwd);
  m.def("grouped_gemm_dgrad", &grouped_gemm_dgrad);
  m.def("grouped_gemm_wgrad", &grouped_gemm_wgrad);
  m.def("topk_router", &topk_router);
  m.def("lm_head_splits", &lm_head_splits);
  m.def("lm_head_logprob", &lm_head_logprob);
  m.def("lm_head_dlogits", &lm_head_dlogits);
}
