// Bindings of what the rollout engine's serving path launches: matrix products, prefill attention, sampling, the decode
// advance, and the kernels of composed stacks.  They are part of the full extension and, alone, of the small
// serving extension (module_serving.cpp).
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include "api.h"
#include "host_utils.h"

namespace {
// Also clears this thread's "last error" slot (an unrelated, already handled status must not look like a launch failure).
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
inline const void* optptr(const c10::optional<torch::Tensor>& t) { return t.has_value() ? t->data_ptr() : nullptr; }
inline const int* optint(const c10::optional<torch::Tensor>& t) { return t.has_value() ? t->data_ptr<int>() : nullptr; }
// composed stacks run in bf16 or in fp32
inline int is_fp32(const torch::Tensor& t) {
  TORCH_CHECK(t.scalar_type() == at::kFloat || t.scalar_type() == at::kBFloat16, "bf16 or fp32 expected, got ", t.scalar_type());
  return t.scalar_type() == at::kFloat;
}
inline bool is_i32(const torch::Tensor& t) { return t.scalar_type() == at::kInt && t.is_contiguous(); }
inline void check_same(const torch::Tensor& a, const torch::Tensor& b, const char* what) {
  TORCH_CHECK(a.scalar_type() == b.scalar_type() && a.device() == b.device(), what, ": operands differ in type or device");
}

void gemm(torch::Tensor A, torch::Tensor B, torch::Tensor C, c10::optional<torch::Tensor> bias, int64_t M, int64_t N,
          int64_t K, int64_t lda, int64_t ldb, int64_t ldc, bool a_mn, bool b_mn, bool accumulate, int64_t force_bn,
          int64_t lbo_a, int64_t sbo_a, int64_t lbo_b, int64_t sbo_b, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(A.device());
  TORCH_CHECK(A.scalar_type() == B.scalar_type(), "A/B dtype mismatch");
  const bool fp16 = A.scalar_type() == at::kHalf;
  TORCH_CHECK(fp16 || A.scalar_type() == at::kBFloat16, "gemm inputs must be bf16 or fp16");
  const bool out_fp32 = C.scalar_type() == at::kFloat;
  TORCH_CHECK(out_fp32 || C.scalar_type() == A.scalar_type(), "output must be fp32 or the input dtype");
  check(rb_gemm(A.data_ptr(), B.data_ptr(), C.data_ptr(), optptr(bias), (int)M, (int)N, (int)K, (int)lda, (int)ldb,
                (int)ldc, a_mn, b_mn, out_fp32, accumulate, fp16, (int)force_bn, (int)lbo_a, (int)sbo_a, (int)lbo_b,
                (int)sbo_b, err.data_ptr<int>(), cur_stream()),
        "rb_gemm");
}
// CTA-pair kernel; returns false when the problem does not qualify (the caller then uses `gemm`).
bool gemm_pair(torch::Tensor A, torch::Tensor B, torch::Tensor C, int64_t M, int64_t N, int64_t K, int64_t lda, int64_t ldb,
               int64_t ldc, bool a_mn, bool b_mn, bool accumulate, int64_t force_bn, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(A.device());
  TORCH_CHECK(A.scalar_type() == at::kBFloat16 && B.scalar_type() == at::kBFloat16, "gemm_pair inputs must be bf16");
  const bool out_fp32 = C.scalar_type() == at::kFloat;
  TORCH_CHECK(out_fp32 || C.scalar_type() == at::kBFloat16, "output must be fp32 or bf16");
  const int rc = rb_gemm_pair(A.data_ptr(), B.data_ptr(), C.data_ptr(), (int)M, (int)N, (int)K, (int)lda, (int)ldb, (int)ldc,
                              a_mn, b_mn, out_fp32, accumulate, (int)force_bn, err.data_ptr<int>(), cur_stream());
  if (rc == -20) return false;
  check(rc, "rb_gemm_pair");
  return true;
}
void fa_fwd(torch::Tensor q, torch::Tensor k, torch::Tensor v, torch::Tensor o, torch::Tensor lse, torch::Tensor cu_q,
            torch::Tensor cu_k, int64_t max_q_blocks, bool causal, double scale, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(q.device());
  TORCH_CHECK(q.scalar_type() == at::kBFloat16 && q.size(2) == 128, "flash attention: bf16, head_dim 128");
  TORCH_CHECK(q.stride(2) == 1 && k.stride(2) == 1 && v.stride(2) == 1, "head dimension must be contiguous");
  check(rb_fa_fwd(q.data_ptr(), k.data_ptr(), v.data_ptr(), o.data_ptr(), lse.data_ptr<float>(), cu_q.data_ptr<int>(),
                  cu_k.data_ptr<int>(), (int)cu_q.numel() - 1, (int)q.size(0), (int)k.size(0), (int)q.size(1),
                  (int)k.size(1), q.stride(0), q.stride(1), k.stride(0), k.stride(1), v.stride(0), v.stride(1), causal,
                  (float)scale, (int)max_q_blocks, err.data_ptr<int>(), cur_stream()),
        "rb_fa_fwd");
}
void sample_v2(torch::Tensor logits, torch::Tensor temperature, torch::Tensor top_k, torch::Tensor top_p,
               torch::Tensor uniform, torch::Tensor tok, torch::Tensor logp, int64_t V) {
  const c10::cuda::CUDAGuard guard(logits.device());
  TORCH_CHECK(logits.dim() == 2 && logits.stride(1) == 1, "sample: logits rows must be contiguous");
  const bool bf = logits.scalar_type() == at::kBFloat16;
  TORCH_CHECK(bf || logits.scalar_type() == at::kFloat, "sample: bf16 or fp32 logits");
  check(rb_sample_v2(logits.data_ptr(), bf ? 1 : 0, (int)logits.size(0), (int)V, (long long)logits.stride(0),
                     temperature.data_ptr<float>(), (const long long*)top_k.data_ptr<int64_t>(), top_p.data_ptr<float>(),
                     uniform.data_ptr<float>(), (long long*)tok.data_ptr<int64_t>(), logp.data_ptr<float>(), cur_stream()),
        "rb_sample_v2");
}
void decode_advance(torch::Tensor tok_new, torch::Tensor lp_new, torch::Tensor tok_in, torch::Tensor pos, torch::Tensor ctx,
                    torch::Tensor slot, torch::Tensor block_table, int64_t block_size, torch::Tensor active,
                    torch::Tensor remain, torch::Tensor eos, torch::Tensor stop_ids, torch::Tensor out_tok,
                    torch::Tensor out_lp, torch::Tensor counter, torch::Tensor u_all, torch::Tensor u_next) {
  const c10::cuda::CUDAGuard guard(tok_new.device());
  const int B = (int)tok_in.size(0);
  TORCH_CHECK(block_table.dim() == 2 && block_table.size(0) == B && block_table.is_contiguous(), "block table [B, max_blocks]");
  TORCH_CHECK(out_tok.dim() == 2 && out_tok.size(1) == B && out_tok.is_contiguous() && out_lp.is_contiguous(), "window ring [W, B]");
  TORCH_CHECK(u_all.dim() == 2 && u_all.size(0) == out_tok.size(0) && u_all.size(1) == B && u_all.is_contiguous(), "u_all [W, B]");
  TORCH_CHECK(stop_ids.dim() == 2 && stop_ids.size(0) == B && stop_ids.is_contiguous(), "stop ids [B, n]");
  check(rb_decode_advance((const long long*)tok_new.data_ptr<int64_t>(), lp_new.data_ptr<float>(),
                          (long long*)tok_in.data_ptr<int64_t>(), (long long*)pos.data_ptr<int64_t>(), ctx.data_ptr<int>(),
                          (long long*)slot.data_ptr<int64_t>(), block_table.data_ptr<int>(), (int)block_table.size(1),
                          (int)block_size, active.data_ptr<int>(), remain.data_ptr<int>(),
                          (const long long*)eos.data_ptr<int64_t>(), (const long long*)stop_ids.data_ptr<int64_t>(),
                          (int)stop_ids.size(1), (long long*)out_tok.data_ptr<int64_t>(), out_lp.data_ptr<float>(),
                          counter.data_ptr<int>(), (int)out_tok.size(0), u_all.data_ptr<float>(), u_next.data_ptr<float>(), B,
                          cur_stream()),
        "rb_decode_advance");
}
// Weight-streaming decode GEMM; returns false when the shape is outside its range (the caller uses the split-K path).
bool decode_gemm(torch::Tensor x, torch::Tensor W, torch::Tensor y, int64_t glu, int64_t splits, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(x.device());
  TORCH_CHECK(x.scalar_type() == at::kBFloat16 && W.scalar_type() == at::kBFloat16, "bf16 only");
  TORCH_CHECK(y.scalar_type() == (glu == 4 ? at::kFloat : at::kBFloat16), "decode_gemm: output type");
  TORCH_CHECK(x.dim() == 2 && W.dim() == 2 && x.stride(1) == 1 && W.stride(1) == 1 && y.is_contiguous(), "row-major operands");
  const int rc = rb_decode_gemm(x.data_ptr(), W.data_ptr(), y.data_ptr(), (int)x.size(0), (int)W.size(0), (int)x.size(1),
                                (int)x.stride(0), (int)W.stride(0), (int)glu, (int)splits, err.data_ptr<int>(), cur_stream());
  if (rc == -20) return false;
  check(rc, "rb_decode_gemm");
  return true;
}
std::tuple<int64_t, int64_t> gemm_splitk_plan(int64_t M, int64_t N, int64_t K) {
  int bn = 0;
  const int s = rb_gemm_splitk_plan((int)M, (int)N, (int)K, &bn);
  return {s, bn};
}
void gemm_splitk(torch::Tensor A, torch::Tensor B, torch::Tensor C, c10::optional<torch::Tensor> bias,
                 c10::optional<torch::Tensor> residual, torch::Tensor workspace, int64_t splits, int64_t bn,
                 torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(A.device());
  check(rb_gemm_splitk(A.data_ptr(), B.data_ptr(), C.data_ptr(), bias.has_value() ? bias->data_ptr() : nullptr,
                       residual.has_value() ? residual->data_ptr() : nullptr, workspace.data_ptr<float>(), (int)A.size(0),
                       (int)B.size(0), (int)A.size(1), (int)A.stride(0), (int)B.stride(0), (int)C.stride(0), (int)splits,
                       (int)bn, A.scalar_type() == at::kHalf, err.data_ptr<int>(), cur_stream()),
        "rb_gemm_splitk");
}

// ---- composed stacks
void embed_rows(torch::Tensor tok, torch::Tensor w, torch::Tensor res, torch::Tensor h, double scale) {
  const c10::cuda::CUDAGuard guard(w.device());
  check_same(w, h, "embed_rows");
  TORCH_CHECK(tok.scalar_type() == at::kLong && tok.is_contiguous() && w.is_contiguous() && res.is_contiguous() && h.is_contiguous());
  TORCH_CHECK(res.scalar_type() == at::kFloat && res.sizes() == h.sizes() && h.size(0) == tok.numel() && h.size(1) == w.size(1));
  check(rb_embed_rows((const long long*)tok.data_ptr<int64_t>(), w.data_ptr(), res.data_ptr<float>(), h.data_ptr(), (int)tok.numel(),
                      (int)w.size(0), (int)w.size(1), (float)scale, is_fp32(w), cur_stream()),
        "rb_embed_rows");
}
void norm_add(torch::Tensor res, torch::Tensor y, torch::Tensor w, c10::optional<torch::Tensor> next_w, torch::Tensor h, int64_t width,
              int64_t groups, double eps) {
  const c10::cuda::CUDAGuard guard(res.device());
  check_same(y, w, "norm_add");
  check_same(y, h, "norm_add");
  TORCH_CHECK(res.scalar_type() == at::kFloat && res.is_contiguous() && h.is_contiguous() && res.sizes() == h.sizes());
  TORCH_CHECK(y.dim() == 2 && y.stride(1) == 1 && y.size(0) == res.size(0) && y.size(1) >= width && w.numel() == res.size(1));
  TORCH_CHECK(!next_w.has_value() || (next_w->numel() == w.numel() && next_w->scalar_type() == w.scalar_type()));
  TORCH_CHECK(reinterpret_cast<uintptr_t>(y.data_ptr()) % 16 == 0, "norm_add: unaligned input");
  check(rb_norm_add(res.data_ptr<float>(), y.data_ptr(), w.data_ptr(), optptr(next_w), h.data_ptr(), (int)res.size(0), (int)y.stride(0),
                    (int)res.size(1), (int)width, (int)groups, (float)eps, is_fp32(y), cur_stream()),
        "rb_norm_add");
}
// Returns false when `o_raw` is not given and the shape is outside what the tensor-core kernel takes.
bool hgrn2(torch::Tensor qfv, torch::Tensor f_bias, torch::Tensor lower, torch::Tensor norm_w, torch::Tensor state, torch::Tensor slot,
           torch::Tensor ctx, c10::optional<torch::Tensor> cu, c10::optional<torch::Tensor> o_raw, c10::optional<torch::Tensor> spans,
           c10::optional<torch::Tensor> first, c10::optional<torch::Tensor> span_state, c10::optional<torch::Tensor> span_gate,
           torch::Tensor out, int64_t dim, int64_t vdim, double eps) {
  const c10::cuda::CUDAGuard guard(qfv.device());
  for (const auto& t : {f_bias, lower, norm_w, out}) check_same(qfv, t, "hgrn2");
  const int64_t H = state.size(1), rows = qfv.size(0), segs = slot.numel();
  TORCH_CHECK(state.dim() == 4 && state.scalar_type() == at::kFloat && state.is_contiguous() && state.size(2) == dim, "hgrn2: state");
  TORCH_CHECK(qfv.dim() == 2 && qfv.stride(1) == 1 && out.is_contiguous() && out.size(0) == rows, "hgrn2: rows");
  TORCH_CHECK(f_bias.numel() == H * dim && lower.numel() == H * dim && norm_w.numel() == vdim && f_bias.is_contiguous() && lower.is_contiguous());
  TORCH_CHECK(slot.scalar_type() == at::kInt && ctx.scalar_type() == at::kInt && ctx.numel() == segs && slot.is_contiguous() && ctx.is_contiguous());
  if (cu.has_value()) {
    TORCH_CHECK(cu->scalar_type() == at::kInt && cu->numel() == segs + 1 && cu->is_contiguous());
    if (!o_raw.has_value()) {      // tensor-core chunks (bf16)
      TORCH_CHECK(qfv.scalar_type() == at::kBFloat16, "hgrn2: the 32-bit scan needs its scratch");
      const int64_t n = spans.has_value() ? spans->size(0) : 0;
      if (n) {
        TORCH_CHECK(spans->scalar_type() == at::kInt && spans->dim() == 2 && spans->size(1) == 2 && spans->is_contiguous());
        TORCH_CHECK(first.has_value() && first->scalar_type() == at::kInt && first->numel() == segs + 1 && first->is_contiguous());
        TORCH_CHECK(span_state.has_value() && span_state->scalar_type() == at::kFloat && span_state->numel() >= n * state.stride(0));
        TORCH_CHECK(span_gate.has_value() && span_gate->scalar_type() == at::kFloat && span_gate->numel() >= n * H * dim);
      }
      const int rc = rb_hgrn2_chunk(qfv.data_ptr(), f_bias.data_ptr(), lower.data_ptr(), norm_w.data_ptr(), state.data_ptr<float>(),
                                    slot.data_ptr<int>(), ctx.data_ptr<int>(), cu->data_ptr<int>(), n ? spans->data_ptr<int>() : nullptr,
                                    n ? first->data_ptr<int>() : nullptr, n ? span_state->data_ptr<float>() : nullptr,
                                    n ? span_gate->data_ptr<float>() : nullptr, out.data_ptr(), (int)rows, (int)segs, (int)n, (int)H, (int)dim, (int)vdim, (int)state.size(3), (int)qfv.stride(0), (int)out.size(1), (float)eps, cur_stream());
      if (rc == -20) return false;
      check(rc, "rb_hgrn2_chunk");
      return true;
    }
    TORCH_CHECK(o_raw.has_value() && o_raw->scalar_type() == at::kFloat && o_raw->numel() >= rows * H * vdim);
  } else {
    TORCH_CHECK(segs == rows, "hgrn2: one row per segment");
  }
  check(rb_hgrn2(qfv.data_ptr(), f_bias.data_ptr(), lower.data_ptr(), norm_w.data_ptr(), state.data_ptr<float>(), slot.data_ptr<int>(),
                 ctx.data_ptr<int>(), optint(cu), o_raw.has_value() ? o_raw->data_ptr<float>() : nullptr, out.data_ptr(), (int)rows, (int)segs,
                 (int)H, (int)dim, (int)vdim, (int)state.size(3), (int)qfv.stride(0), (int)out.size(1), (float)eps, is_fp32(qfv), cur_stream()),
        "rb_hgrn2");
  return true;
}
// k_rot, q, table: the rotated key part and the query heads [T][H][dk] (features dim .. dim + rot turn in place) of the same projection
void latent_write(torch::Tensor raw, c10::optional<torch::Tensor> k_rot, c10::optional<torch::Tensor> q, c10::optional<torch::Tensor> table, torch::Tensor w,
                  torch::Tensor pool, torch::Tensor slots, int64_t rank, int64_t part, int64_t rot, int64_t dim, double eps) {
  const c10::cuda::CUDAGuard guard(raw.device());
  TORCH_CHECK(rot == 0 || (k_rot.has_value() && q.has_value() && table.has_value()), "latent_write: rotated parts");
  if (rot) {
    check_same(raw, *k_rot, "latent_write");
    check_same(raw, *q, "latent_write");
    const bool one = raw.size(0) == 1;      // (a dimension of size one may have any stride)
    TORCH_CHECK(k_rot->dim() == 2 && (one || k_rot->stride(0) == raw.stride(0)) && k_rot->stride(1) == 1 && k_rot->size(1) >= rot &&
                k_rot->size(0) == raw.size(0), "latent_write: rotated key part");
    TORCH_CHECK(q->dim() == 3 && q->size(0) == raw.size(0) && (one || q->stride(0) == raw.stride(0)) && q->stride(2) == 1 &&
                (q->size(1) == 1 || q->stride(1) == q->size(2)), "latent_write: queries");
    TORCH_CHECK(table->scalar_type() == at::kFloat && table->is_contiguous() && table->numel() == raw.size(0) * rot, "latent_write: angles");
  }
  check_same(raw, w, "latent_write");
  check_same(raw, pool, "latent_write");
  TORCH_CHECK(raw.dim() == 2 && raw.stride(1) == 1 && raw.size(1) >= rank && w.numel() >= rank && pool.dim() == 2 && pool.is_contiguous());
  TORCH_CHECK(slots.scalar_type() == at::kLong && slots.is_contiguous() && slots.numel() == raw.size(0));
  check(rb_latent_write(raw.data_ptr(), rot ? k_rot->data_ptr() : nullptr, rot ? q->data_ptr() : nullptr, (int)raw.stride(0), w.data_ptr(), pool.data_ptr(),
                        (const long long*)slots.data_ptr<int64_t>(), rot ? table->data_ptr<float>() : nullptr, pool.size(0), (int)raw.size(0), (int)rank,
                        (int)pool.size(1), (int)part, (int)rot, rot ? (int)q->size(1) : 0, rot ? (int)q->size(2) : 0, (int)dim, (float)eps, is_fp32(raw),
                        cur_stream()),
        "rb_latent_write");
}
void latent_attn(torch::Tensor q, torch::Tensor pool, torch::Tensor bt, c10::optional<torch::Tensor> row_seg, c10::optional<torch::Tensor> row_pos,
                 torch::Tensor ctx, c10::optional<torch::Tensor> gate, torch::Tensor out, int64_t block_size, double scale) {
  const c10::cuda::CUDAGuard guard(q.device());
  check_same(q, pool, "latent_attn");
  check_same(q, out, "latent_attn");
  const int64_t T = q.size(0);
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && out.dim() == 3 && out.is_contiguous() && pool.is_contiguous() && pool.size(1) == q.size(2));
  TORCH_CHECK(out.size(0) == T && out.size(1) == q.size(1) && out.size(2) <= q.size(2), "latent_attn: output");
  TORCH_CHECK(bt.scalar_type() == at::kInt && bt.is_contiguous() && ctx.scalar_type() == at::kInt && ctx.is_contiguous());
  TORCH_CHECK(row_seg.has_value() == row_pos.has_value());
  TORCH_CHECK(row_seg.has_value() ? (row_seg->numel() == T && row_pos->numel() == T && row_seg->scalar_type() == at::kInt &&
                                     row_pos->scalar_type() == at::kInt)
                                  : (ctx.numel() == T && bt.size(0) == T), "latent_attn: row description");
  TORCH_CHECK(!gate.has_value() || (gate->scalar_type() == q.scalar_type() && gate->stride(1) == 1 && gate->size(0) == T));
  check(rb_latent_attn(q.data_ptr(), pool.data_ptr(), bt.data_ptr<int>(), optint(row_seg), optint(row_pos), ctx.data_ptr<int>(), optptr(gate),
                       out.data_ptr(), (int)T, (int)q.size(1), (int)q.size(2), (int)out.size(2), (int)bt.size(1), (int)block_size,
                       gate.has_value() ? (int)gate->stride(0) : 0, (float)scale, is_fp32(q), cur_stream()),
        "rb_latent_attn");
}
// Tensor-core form (bf16); returns false for shapes it does not take (the caller then uses latent_attn).
bool latent_attn_tc(torch::Tensor q, torch::Tensor pool, torch::Tensor bt, c10::optional<torch::Tensor> items, torch::Tensor ctx,
                    c10::optional<torch::Tensor> gate, torch::Tensor out, c10::optional<torch::Tensor> part_o,
                    c10::optional<torch::Tensor> part_ml, int64_t block_size, int64_t width, int64_t splits, double scale, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(q.device());
  const int64_t T = q.size(0), H = q.size(1), R = q.size(2), Rv = out.size(2);
  TORCH_CHECK(q.scalar_type() == at::kBFloat16 && pool.scalar_type() == at::kBFloat16 && out.scalar_type() == at::kBFloat16);
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && out.dim() == 3 && out.is_contiguous() && pool.is_contiguous() && pool.size(1) == R);
  TORCH_CHECK(out.size(0) == T && out.size(1) == H && Rv <= R, "latent_attn_tc: output");
  TORCH_CHECK(bt.scalar_type() == at::kInt && bt.is_contiguous() && ctx.scalar_type() == at::kInt && ctx.is_contiguous());
  if (items.has_value()) {
    TORCH_CHECK(items->scalar_type() == at::kInt && items->dim() == 2 && items->size(1) == 4 && items->is_contiguous());
  } else {
    TORCH_CHECK(ctx.numel() == T && bt.size(0) == T, "latent_attn_tc: one row per segment");
  }
  TORCH_CHECK(!gate.has_value() || (gate->scalar_type() == at::kBFloat16 && gate->stride(1) == 1 && gate->size(0) == T));
  TORCH_CHECK(splits == 1 || (part_o.has_value() && part_o->numel() >= splits * T * H * Rv && part_ml.has_value() &&
                              part_ml->numel() >= splits * T * H * 2), "latent_attn_tc: scratch");
  const int rc = rb_latent_attn_tc(q.data_ptr(), pool.data_ptr(), bt.data_ptr<int>(), optint(items), ctx.data_ptr<int>(), optptr(gate), out.data_ptr(),
                                   part_o.has_value() ? part_o->data_ptr<float>() : nullptr, part_ml.has_value() ? part_ml->data_ptr<float>() : nullptr,
                                   (int)T, (int)H, (int)R, (int)Rv, pool.size(0), (int)bt.size(1), (int)block_size,
                                   items.has_value() ? (int)items->size(0) : 0, (int)width, (int)splits,
                                   gate.has_value() ? (int)gate->stride(0) : 0, (float)scale, err.data_ptr<int>(), cur_stream());
  if (rc == -20) return false;
  check(rc, "rb_latent_attn_tc");
  return true;
}
// gate: columns of a gate per output feature, [T, >= H N], or none
inline int gate_pitch(const c10::optional<torch::Tensor>& gate, const torch::Tensor& like, int64_t rows, int64_t cols) {
  if (!gate.has_value()) return 0;
  TORCH_CHECK(gate->scalar_type() == like.scalar_type() && gate->device() == like.device() && gate->dim() == 2 && gate->stride(1) == 1, "output gate: layout");
  TORCH_CHECK(gate->size(0) == rows && gate->size(1) >= cols, "output gate: shape");
  return (int)gate->stride(0);
}
bool head_gemm(torch::Tensor x, torch::Tensor w, c10::optional<torch::Tensor> gate, torch::Tensor out, bool kn, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(x.device());
  TORCH_CHECK(x.scalar_type() == at::kBFloat16 && w.scalar_type() == at::kBFloat16 && out.scalar_type() == at::kBFloat16);
  TORCH_CHECK(x.dim() == 3 && w.dim() == 3 && out.dim() == 3 && x.stride(2) == 1 && w.is_contiguous() && out.is_contiguous());
  TORCH_CHECK(w.size(0) == x.size(1) && w.size(kn ? 1 : 2) == x.size(2) && out.size(0) == x.size(0) && out.size(1) == x.size(1) &&
              out.size(2) == w.size(kn ? 2 : 1), "head_gemm: shapes");
  const int rc = rb_head_gemm(x.data_ptr(), w.data_ptr(), optptr(gate), gate_pitch(gate, x, x.size(0), out.size(1) * out.size(2)), out.data_ptr(), (int)x.size(0), (int)x.size(1), (int)out.size(2), (int)x.size(2), x.stride(0),
                              x.stride(1), kn, err.data_ptr<int>(), cur_stream());
  if (rc == -20) return false;
  check(rc, "rb_head_gemm");
  return true;
}
// o [T, ...] times the sigmoid of a gate per feature, in place
void gate_outputs(torch::Tensor o, torch::Tensor gate) {
  const c10::cuda::CUDAGuard guard(o.device());
  TORCH_CHECK(o.is_contiguous() && o.size(0) > 0, "gate_outputs: layout");
  const int64_t n = o.numel() / o.size(0);
  const int ld = gate_pitch(gate, o, o.size(0), n);
  check(rb_gate_outputs(o.data_ptr(), gate.data_ptr(), ld, (int)o.size(0), (int)n, is_fp32(o), cur_stream()), "rb_gate_outputs");
}
void glu(torch::Tensor in, torch::Tensor out, int64_t act) {
  const c10::cuda::CUDAGuard guard(in.device());
  check_same(in, out, "glu");
  TORCH_CHECK(in.dim() == 2 && in.stride(1) == 1 && out.is_contiguous() && in.size(1) == 2 * out.size(1) && in.size(0) == out.size(0));
  check(rb_glu(in.data_ptr(), out.data_ptr(), in.size(0), (int)out.size(1), (int)in.stride(0), (int)act, is_fp32(in), cur_stream()), "rb_glu");
}
// C[z] = A[z] op(B[z]) on CUDA cores; every operand [batch, rows, cols] with unit inner stride.
void simt_gemm(torch::Tensor A, torch::Tensor B, torch::Tensor C, bool b_kn) {
  const c10::cuda::CUDAGuard guard(A.device());
  check_same(A, B, "simt_gemm");
  check_same(A, C, "simt_gemm");
  TORCH_CHECK(A.dim() == 3 && B.dim() == 3 && C.dim() == 3 && A.stride(2) == 1 && B.stride(2) == 1 && C.stride(2) == 1);
  const int64_t K = A.size(2), N = C.size(2);
  TORCH_CHECK(A.size(0) == C.size(0) && B.size(0) == C.size(0) && A.size(1) == C.size(1) && B.size(1) == (b_kn ? K : N) && B.size(2) == (b_kn ? N : K),
              "simt_gemm: shapes");
  check(rb_simt_gemm(A.data_ptr(), B.data_ptr(), C.data_ptr(), (int)A.size(1), (int)N, (int)K, (int)A.stride(1), (int)B.stride(1), (int)C.stride(1),
                     b_kn, (int)A.size(0), A.stride(0), B.stride(0), C.stride(0), is_fp32(A), cur_stream()),
        "rb_simt_gemm");
}
// ---- attention over cached keys and values, routed experts
void embed_norm(torch::Tensor tok, torch::Tensor table, torch::Tensor w, torch::Tensor res, torch::Tensor h, int64_t width, int64_t groups, double eps) {
  const c10::cuda::CUDAGuard guard(table.device());
  check_same(table, h, "embed_norm");
  check_same(table, w, "embed_norm");
  TORCH_CHECK(tok.scalar_type() == at::kLong && tok.is_contiguous() && table.is_contiguous() && res.is_contiguous() && h.is_contiguous());
  TORCH_CHECK(res.scalar_type() == at::kFloat && res.sizes() == h.sizes() && h.size(0) == tok.numel() && h.size(1) == table.size(1) && w.numel() == table.size(1));
  check(rb_embed_norm((const long long*)tok.data_ptr<int64_t>(), table.data_ptr(), w.data_ptr(), res.data_ptr<float>(), h.data_ptr(), (int)tok.numel(),
                      (int)table.size(0), (int)table.size(1), (int)width, (int)groups, (float)eps, is_fp32(table), cur_stream()),
        "rb_embed_norm");
}
// choices from `experts` on (= entries of offset - 1) are identity experts
inline int check_experts(const torch::Tensor& res, const torch::Tensor& ex, const torch::Tensor& expert, const torch::Tensor& place,
                         const torch::Tensor& offset, const torch::Tensor& weight) {
  TORCH_CHECK(ex.dim() == 2 && ex.is_contiguous() && ex.size(1) == res.size(1) && ex.size(0) == expert.numel(), "expert rows");
  TORCH_CHECK(is_i32(expert) && is_i32(place) && is_i32(offset) && weight.scalar_type() == at::kFloat && weight.is_contiguous(), "expert plan: types");
  TORCH_CHECK(expert.dim() == 2 && expert.size(0) == res.size(0) && place.sizes() == expert.sizes() && weight.sizes() == expert.sizes(), "expert plan: shapes");
  return (int)offset.numel() - 1;
}
// x <- norm(alpha x + y + weighted expert rows); y or the experts may be missing.  centre: layer norm (bias b), else RMS.  next_w: h is the
// norm of the new stream with it, times scale.
void sum_norm(torch::Tensor res, c10::optional<torch::Tensor> y, c10::optional<torch::Tensor> ex, c10::optional<torch::Tensor> expert,
              c10::optional<torch::Tensor> place, c10::optional<torch::Tensor> offset, c10::optional<torch::Tensor> weight, torch::Tensor w,
              c10::optional<torch::Tensor> b, c10::optional<torch::Tensor> next_w, c10::optional<torch::Tensor> next_b, torch::Tensor h, int64_t width,
              bool centre, double alpha, double eps, double scale) {
  const c10::cuda::CUDAGuard guard(res.device());
  check_same(w, h, "sum_norm");
  TORCH_CHECK(res.scalar_type() == at::kFloat && res.is_contiguous() && h.is_contiguous() && res.sizes() == h.sizes() && w.numel() == res.size(1));
  for (const auto& t : {b, next_w, next_b})
    if (t.has_value()) {
      check_same(w, *t, "sum_norm");
      TORCH_CHECK(t->numel() == w.numel() && t->is_contiguous(), "sum_norm: weights");
    }
  if (y.has_value()) {
    check_same(w, *y, "sum_norm");
    TORCH_CHECK(y->is_contiguous() && y->sizes() == res.sizes(), "sum_norm: input");
  }
  int top = 0, experts = 0;
  if (ex.has_value()) {
    check_same(w, *ex, "sum_norm");
    TORCH_CHECK(expert.has_value() && place.has_value() && offset.has_value() && weight.has_value(), "sum_norm: expert plan");
    experts = check_experts(res, *ex, *expert, *place, *offset, *weight);
    top = (int)expert->size(1);
  }
  check(rb_sum_norm(res.data_ptr<float>(), optptr(y), optptr(ex), optint(expert), optint(place), optint(offset),
                    weight.has_value() ? weight->data_ptr<float>() : nullptr, top, experts, w.data_ptr(), optptr(b), optptr(next_w), optptr(next_b), h.data_ptr(),
                    (int)res.size(0), (int)res.size(1), (int)res.size(1), (int)width, centre, (float)alpha, (float)eps, (float)scale, is_fp32(w), cur_stream()),
        "rb_sum_norm");
}
void norm_add_experts(torch::Tensor res, c10::optional<torch::Tensor> y, torch::Tensor ex, torch::Tensor expert, torch::Tensor place, torch::Tensor offset,
                      torch::Tensor weight, torch::Tensor w, c10::optional<torch::Tensor> next_w, torch::Tensor h, int64_t width, int64_t groups, double eps) {
  const c10::cuda::CUDAGuard guard(res.device());
  check_same(ex, w, "norm_add_experts");
  check_same(ex, h, "norm_add_experts");
  TORCH_CHECK(res.scalar_type() == at::kFloat && res.is_contiguous() && h.is_contiguous() && res.sizes() == h.sizes() && w.numel() == res.size(1));
  const int experts = check_experts(res, ex, expert, place, offset, weight);
  TORCH_CHECK(!y.has_value() || (y->scalar_type() == ex.scalar_type() && y->is_contiguous() && y->sizes() == res.sizes()));
  TORCH_CHECK(!next_w.has_value() || (next_w->numel() == w.numel() && next_w->scalar_type() == w.scalar_type()));
  check(rb_norm_add_experts(res.data_ptr<float>(), optptr(y), ex.data_ptr(), expert.data_ptr<int>(), place.data_ptr<int>(), offset.data_ptr<int>(),
                            weight.data_ptr<float>(), (int)expert.size(1), experts, w.data_ptr(), optptr(next_w), h.data_ptr(), (int)res.size(0),
                            (int)ex.size(1), (int)res.size(1), (int)width, (int)groups, (float)eps, is_fp32(ex), cur_stream()),
        "rb_norm_add_experts");
}
void rope_table(torch::Tensor pos, int64_t offset, torch::Tensor freq, torch::Tensor out) {
  const c10::cuda::CUDAGuard guard(pos.device());
  TORCH_CHECK(is_i32(pos) && freq.scalar_type() == at::kDouble && freq.is_contiguous() && out.scalar_type() == at::kFloat && out.is_contiguous());
  TORCH_CHECK(out.numel() == pos.numel() * freq.numel() * 2 && freq.device() == pos.device());
  check(rb_rope_table(pos.data_ptr<int>(), (int)offset, freq.data_ptr<double>(), out.data_ptr<float>(), (int)pos.numel(), (int)freq.numel(), cur_stream()),
        "rb_rope_table");
}
void attention_inputs(torch::Tensor qkv, c10::optional<torch::Tensor> table, torch::Tensor q, c10::optional<torch::Tensor> k_pool,
                      c10::optional<torch::Tensor> v_pool, torch::Tensor slots, int64_t kv_heads, int64_t dim, int64_t vdim, int64_t rot, double eps) {
  const c10::cuda::CUDAGuard guard(qkv.device());
  check_same(qkv, q, "attention_inputs");
  const int64_t T = qkv.size(0);
  TORCH_CHECK(qkv.dim() == 2 && qkv.stride(1) == 1 && q.dim() == 3 && q.is_contiguous() && q.size(0) == T && k_pool.has_value() == v_pool.has_value());
  TORCH_CHECK(qkv.size(1) >= q.size(1) * dim + (k_pool.has_value() ? kv_heads * (dim + vdim) : 0), "attention_inputs: columns");
  TORCH_CHECK(rot == 0 || (table.has_value() && table->scalar_type() == at::kFloat && table->is_contiguous() && table->numel() == T * rot));
  TORCH_CHECK(slots.scalar_type() == at::kLong && slots.is_contiguous() && slots.numel() == T);
  if (k_pool.has_value()) {
    check_same(qkv, *k_pool, "attention_inputs");
    check_same(qkv, *v_pool, "attention_inputs");
    TORCH_CHECK(k_pool->dim() == 3 && v_pool->dim() == 3 && k_pool->is_contiguous() && v_pool->is_contiguous() && k_pool->size(0) == v_pool->size(0));
    TORCH_CHECK(k_pool->size(1) == kv_heads && v_pool->size(1) == kv_heads && k_pool->size(2) == q.size(2), "attention_inputs: pools");
  }
  check(rb_attention_inputs(qkv.data_ptr(), (int)qkv.stride(0), rot ? table->data_ptr<float>() : nullptr, q.data_ptr(),
                            k_pool.has_value() ? k_pool->data_ptr() : nullptr, v_pool.has_value() ? v_pool->data_ptr() : nullptr,
                            (const long long*)slots.data_ptr<int64_t>(), k_pool.has_value() ? k_pool->size(0) : 0, (int)T, (int)q.size(1), (int)kv_heads,
                            (int)dim, (int)vdim, (int)q.size(2), v_pool.has_value() ? (int)v_pool->size(2) : 0, (int)rot, (float)eps, is_fp32(qkv),
                            cur_stream()),
        "rb_attention_inputs");
}
// the same with weighted norms over the whole query and key projections (q_w, k_w; none: no norm when eps <= 0); halves: pairs rot / 2 apart
void projection_inputs(torch::Tensor qkv, c10::optional<torch::Tensor> q_w, c10::optional<torch::Tensor> k_w, c10::optional<torch::Tensor> table, torch::Tensor q,
                       c10::optional<torch::Tensor> k_pool, c10::optional<torch::Tensor> v_pool, torch::Tensor slots, int64_t kv_heads, int64_t dim, int64_t vdim,
                       int64_t rot, bool halves, double eps) {
  const c10::cuda::CUDAGuard guard(qkv.device());
  check_same(qkv, q, "projection_inputs");
  const int64_t T = qkv.size(0);
  TORCH_CHECK(qkv.dim() == 2 && qkv.stride(1) == 1 && q.dim() == 3 && q.is_contiguous() && q.size(0) == T && k_pool.has_value() == v_pool.has_value());
  TORCH_CHECK(qkv.size(1) >= q.size(1) * dim + (k_pool.has_value() ? kv_heads * (dim + vdim) : 0), "projection_inputs: columns");
  TORCH_CHECK(rot == 0 || (table.has_value() && table->scalar_type() == at::kFloat && table->is_contiguous() && table->numel() == T * rot));
  TORCH_CHECK(slots.scalar_type() == at::kLong && slots.is_contiguous() && slots.numel() == T);
  if (q_w.has_value()) {
    check_same(qkv, *q_w, "projection_inputs");
    TORCH_CHECK(q_w->is_contiguous() && q_w->numel() == q.size(1) * dim, "projection_inputs: query norm");
  }
  if (k_pool.has_value()) {
    check_same(qkv, *k_pool, "projection_inputs");
    check_same(qkv, *v_pool, "projection_inputs");
    TORCH_CHECK(k_pool->dim() == 3 && v_pool->dim() == 3 && k_pool->is_contiguous() && v_pool->is_contiguous() && k_pool->size(0) == v_pool->size(0));
    TORCH_CHECK(k_pool->size(1) == kv_heads && v_pool->size(1) == kv_heads && k_pool->size(2) == q.size(2), "projection_inputs: pools");
    if (k_w.has_value()) {
      check_same(qkv, *k_w, "projection_inputs");
      TORCH_CHECK(k_w->is_contiguous() && k_w->numel() == kv_heads * dim, "projection_inputs: key norm");
    }
  }
  check(rb_projection_inputs(qkv.data_ptr(), (int)qkv.stride(0), optptr(q_w), optptr(k_w), rot ? table->data_ptr<float>() : nullptr, q.data_ptr(),
                             k_pool.has_value() ? k_pool->data_ptr() : nullptr, v_pool.has_value() ? v_pool->data_ptr() : nullptr,
                             (const long long*)slots.data_ptr<int64_t>(), k_pool.has_value() ? k_pool->size(0) : 0, (int)T, (int)q.size(1), (int)kv_heads,
                             (int)dim, (int)vdim, (int)q.size(2), v_pool.has_value() ? (int)v_pool->size(2) : 0, (int)rot, halves, (float)eps, is_fp32(qkv),
                             cur_stream()),
        "rb_projection_inputs");
}
inline void check_pools(const torch::Tensor& q, const torch::Tensor& k, const torch::Tensor& v, const torch::Tensor& bt, const torch::Tensor& ctx,
                        const c10::optional<torch::Tensor>& sink, const torch::Tensor& out, bool wide = false) {
  check_same(q, k, "paged attention");
  check_same(q, v, "paged attention");
  check_same(q, out, "paged attention");
  TORCH_CHECK(q.dim() == 3 && k.dim() == 3 && v.dim() == 3 && q.is_contiguous() && k.is_contiguous() && v.is_contiguous() && out.is_contiguous());
  TORCH_CHECK(k.size(2) == q.size(2) && v.size(0) == k.size(0) && v.size(1) == k.size(1) && q.size(1) % k.size(1) == 0, "paged attention: shapes");
  const int64_t outs = q.size(1) * (wide ? k.size(1) : 1);      // out: every head's columns, wide: for every group
  TORCH_CHECK(out.dim() == 2 && out.size(0) == q.size(0) && out.size(1) % outs == 0 && out.size(1) / outs <= v.size(2), "paged attention: output");
  TORCH_CHECK(is_i32(bt) && bt.dim() == 2 && is_i32(ctx) && ctx.numel() == bt.size(0), "paged attention: block tables");
  TORCH_CHECK(!sink.has_value() || (sink->scalar_type() == q.scalar_type() && sink->is_contiguous() && sink->numel() == q.size(1)), "paged attention: sink");
}
void gqa_attn(torch::Tensor q, torch::Tensor k, torch::Tensor v, torch::Tensor bt, c10::optional<torch::Tensor> row_seg, c10::optional<torch::Tensor> row_pos,
              torch::Tensor ctx, c10::optional<torch::Tensor> sink, c10::optional<torch::Tensor> gate, torch::Tensor out, int64_t block_size, int64_t window,
              int64_t keep, int64_t chunk, bool wide, double scale, double cap) {
  const c10::cuda::CUDAGuard guard(q.device());
  check_pools(q, k, v, bt, ctx, sink, out, wide);
  const int64_t T = q.size(0), H = q.size(1);
  TORCH_CHECK(row_seg.has_value() == row_pos.has_value());
  TORCH_CHECK(row_seg.has_value() ? (is_i32(*row_seg) && is_i32(*row_pos) && row_seg->numel() == T && row_pos->numel() == T) : ctx.numel() == T,
              "gqa_attn: row description");
  check(rb_gqa_attn(q.data_ptr(), k.data_ptr(), v.data_ptr(), bt.data_ptr<int>(), optint(row_seg), optint(row_pos), ctx.data_ptr<int>(), optptr(sink),
                    optptr(gate), gate_pitch(gate, q, T, out.size(1)), out.data_ptr(), (int)T, (int)H, (int)k.size(1), (int)q.size(2), (int)v.size(2),
                    (int)(out.size(1) / H / (wide ? k.size(1) : 1)), (int)bt.size(1), (int)block_size, (int)window, (int)keep, (int)chunk, wide, (float)scale,
                    (float)cap, is_fp32(q), cur_stream()),
        "rb_gqa_attn");
}
// Prompt portions; returns false for shapes the tensor-core kernel does not take.
bool paged_flash(torch::Tensor q, torch::Tensor k, torch::Tensor v, torch::Tensor bt, torch::Tensor ctx, c10::optional<torch::Tensor> blocks,
                 c10::optional<torch::Tensor> sink, c10::optional<torch::Tensor> gate, torch::Tensor out, int64_t block_size, int64_t window, int64_t keep,
                 int64_t chunk, bool wide, double scale, double cap, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(q.device());
  if (q.scalar_type() != at::kBFloat16) return false;
  check_pools(q, k, v, bt, ctx, sink, out, wide);
  const int64_t T = q.size(0), H = q.size(1);
  TORCH_CHECK(blocks.has_value() ? (is_i32(*blocks) && blocks->dim() == 2 && blocks->size(1) == 4) : ctx.numel() == T, "paged_flash: query tiles");
  const int rc = rb_paged_flash(q.data_ptr(), k.data_ptr(), v.data_ptr(), bt.data_ptr<int>(), ctx.data_ptr<int>(), optint(blocks), optptr(sink),
                                optptr(gate), gate_pitch(gate, q, T, out.size(1)), out.data_ptr(), (int)T, (int)(blocks.has_value() ? blocks->size(0) : T), (int)H, (int)k.size(1), (int)q.size(2), (int)v.size(2),
                                (int)(out.size(1) / H / (wide ? k.size(1) : 1)), k.size(0), (int)block_size, (int)bt.size(1), (int)window, (int)keep, (int)chunk, wide,
                                (float)scale, (float)cap, err.data_ptr<int>(), cur_stream());
  if (rc == -20) return false;
  check(rc, "rb_paged_flash");
  return true;
}
// Keys and values that lie side by side, segment by segment: k, v [rows][H][d], those of segment s from row first[s] on.  q [T][H][dk] may be
// a strided slice.  gate: [T, H] or (features) [T, >= H dv].  Returns false for shapes the kernel does not take.
bool dense_flash(torch::Tensor q, torch::Tensor k, torch::Tensor v, torch::Tensor first, torch::Tensor blocks, c10::optional<torch::Tensor> gate, bool features,
                 torch::Tensor out, double scale, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(q.device());
  if (q.scalar_type() != at::kBFloat16) return false;
  check_same(q, k, "dense_flash");
  check_same(q, v, "dense_flash");
  check_same(q, out, "dense_flash");
  const int64_t T = q.size(0), H = q.size(1);
  TORCH_CHECK(q.dim() == 3 && k.dim() == 3 && v.dim() == 3 && q.stride(2) == 1 && (H == 1 || q.stride(1) == q.size(2)) && k.is_contiguous() && v.is_contiguous());
  TORCH_CHECK(k.size(1) == H && v.size(1) == H && k.size(0) == v.size(0) && k.size(2) == q.size(2), "dense_flash: shapes");
  TORCH_CHECK(out.dim() == 2 && out.is_contiguous() && out.size(0) == T && out.size(1) == H * v.size(2), "dense_flash: output");
  TORCH_CHECK(is_i32(first) && is_i32(blocks) && blocks.dim() == 2 && blocks.size(1) == 4, "dense_flash: tiles");
  const int rc = rb_dense_flash(q.data_ptr(), T > 1 ? q.stride(0) : H * q.size(2), k.data_ptr(), v.data_ptr(), first.data_ptr<int>(), blocks.data_ptr<int>(),
                                optptr(gate), gate_pitch(gate, q, T, features ? out.size(1) : H), !features, out.data_ptr(), (int)T, (int)blocks.size(0), (int)H,
                                (int)q.size(2), (int)v.size(2), k.size(0), (float)scale, err.data_ptr<int>(), cur_stream());
  if (rc == -20) return false;
  check(rc, "rb_dense_flash");
  return true;
}
// One row per sequence; returns false for shapes the tensor-core kernel does not take.
bool paged_decode(torch::Tensor q, torch::Tensor k, torch::Tensor v, torch::Tensor bt, torch::Tensor ctx, c10::optional<torch::Tensor> sink,
                  c10::optional<torch::Tensor> gate, torch::Tensor out, c10::optional<torch::Tensor> part_o, c10::optional<torch::Tensor> part_ml,
                  int64_t block_size, int64_t max_ctx, int64_t window, int64_t keep, int64_t chunk, int64_t splits, double scale, double cap, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(q.device());
  if (q.scalar_type() != at::kBFloat16) return false;
  check_pools(q, k, v, bt, ctx, sink, out);
  const int64_t B = q.size(0), H = q.size(1);
  TORCH_CHECK(ctx.numel() == B, "paged_decode: one row per sequence");
  TORCH_CHECK(splits == 1 || (part_o.has_value() && part_o->scalar_type() == at::kFloat && part_o->numel() >= splits * B * H * 128 && part_ml.has_value() &&
                              part_ml->scalar_type() == at::kFloat && part_ml->numel() >= splits * B * H * 2), "paged_decode: scratch");
  const int rc = rb_paged_decode_tc(q.data_ptr(), k.data_ptr(), v.data_ptr(), bt.data_ptr<int>(), ctx.data_ptr<int>(), optptr(sink), optptr(gate),
                                    gate_pitch(gate, q, B, out.size(1)), out.data_ptr(), part_o.has_value() ? part_o->data_ptr<float>() : nullptr, part_ml.has_value() ? part_ml->data_ptr<float>() : nullptr,
                                    (int)B, (int)H, (int)k.size(1), (int)q.size(2), (int)v.size(2), (int)(out.size(1) / H), k.size(0), (int)block_size,
                                    (int)bt.size(1), (int)max_ctx, (int)window, (int)keep, (int)chunk, (float)scale, (float)cap, (int)splits, err.data_ptr<int>(), cur_stream());
  if (rc == -20) return false;
  check(rc, "rb_paged_decode_tc");
  return true;
}
// (packed head columns, value groups per CTA) of talk_decode for these heads; columns 0: it does not take them
std::tuple<int64_t, int64_t> talk_decode_plan(int64_t H, int64_t G, int64_t dk, int64_t dv) {
  int groups = 0;
  const int cols = rb_talk_decode_plan((int)H, (int)G, (int)dk, (int)dv, &groups);
  return {cols, groups};
}
// One row per sequence with mixed heads; returns false for shapes the kernel does not take.
bool talk_decode(torch::Tensor q, torch::Tensor k, torch::Tensor v, torch::Tensor bt, torch::Tensor ctx, c10::optional<torch::Tensor> sink, torch::Tensor mix,
                 torch::Tensor out, torch::Tensor part_o, torch::Tensor part_l, int64_t block_size, int64_t max_ctx, int64_t window, int64_t keep,
                 int64_t chunk, int64_t splits, double scale, double cap, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(q.device());
  if (q.scalar_type() != at::kBFloat16) return false;
  check_pools(q, k, v, bt, ctx, sink, out);
  check_same(q, mix, "talk_decode");
  const int64_t B = q.size(0), H = q.size(1), G = k.size(1);
  int groups = 0;
  const int64_t cols = rb_talk_decode_plan((int)H, (int)G, (int)q.size(2), (int)v.size(2), &groups);
  if (!cols) return false;
  TORCH_CHECK(ctx.numel() == B && mix.is_contiguous() && mix.numel() == H * H, "talk_decode: one row per sequence");
  TORCH_CHECK(part_o.scalar_type() == at::kFloat && part_o.numel() >= B * splits * G * cols * 128 && part_l.scalar_type() == at::kFloat &&
              part_l.numel() >= B * splits * cols, "talk_decode: scratch");
  const int rc = rb_talk_decode(q.data_ptr(), k.data_ptr(), v.data_ptr(), bt.data_ptr<int>(), ctx.data_ptr<int>(), optptr(sink), mix.data_ptr(), out.data_ptr(),
                                part_o.data_ptr<float>(), part_l.data_ptr<float>(), (int)B, (int)H, (int)G, (int)q.size(2), (int)v.size(2),
                                (int)(out.size(1) / H), k.size(0), (int)block_size, (int)bt.size(1), (int)max_ctx, (int)window, (int)keep, (int)chunk,
                                (float)scale, (float)cap, (int)splits, err.data_ptr<int>(), cur_stream());
  if (rc == -20) return false;
  check(rc, "rb_talk_decode");
  return true;
}
// Prompt portions: every head's weights on every group's values, out [T][H G vo]; returns false for shapes the kernel does not take.
bool talk_flash(torch::Tensor q, torch::Tensor k, torch::Tensor v, torch::Tensor bt, torch::Tensor ctx, c10::optional<torch::Tensor> blocks,
                c10::optional<torch::Tensor> sink, torch::Tensor out, int64_t block_size, int64_t window, int64_t keep, int64_t chunk, double scale, double cap,
                torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(q.device());
  if (q.scalar_type() != at::kBFloat16) return false;
  check_pools(q, k, v, bt, ctx, sink, out, true);
  const int64_t T = q.size(0), H = q.size(1), G = k.size(1);
  TORCH_CHECK(blocks.has_value() ? (is_i32(*blocks) && blocks->dim() == 2 && blocks->size(1) == 4) : ctx.numel() == T, "talk_flash: query tiles");
  const int rc = rb_talk_flash(q.data_ptr(), k.data_ptr(), v.data_ptr(), bt.data_ptr<int>(), ctx.data_ptr<int>(), optint(blocks), optptr(sink), out.data_ptr(),
                               (int)T, (int)(blocks.has_value() ? blocks->size(0) : T), (int)H, (int)G, (int)q.size(2), (int)v.size(2),
                               (int)(out.size(1) / H / G), k.size(0), (int)block_size, (int)bt.size(1), (int)window, (int)keep, (int)chunk, (float)scale,
                               (float)cap, err.data_ptr<int>(), cur_stream());
  if (rc == -20) return false;
  check(rc, "rb_talk_flash");
  return true;
}
// wide [T][H G vo]: what every head's weights make of every group's values; mix [H][H]; out [T][H vo]
void mix_heads(torch::Tensor wide, torch::Tensor mix, torch::Tensor out, int64_t kv_heads) {
  const c10::cuda::CUDAGuard guard(wide.device());
  check_same(wide, mix, "mix_heads");
  check_same(wide, out, "mix_heads");
  const int64_t T = out.size(0), H = mix.size(0);
  TORCH_CHECK(mix.dim() == 2 && mix.size(1) == H && wide.is_contiguous() && mix.is_contiguous() && out.is_contiguous() && out.dim() == 2 && out.size(1) % H == 0);
  TORCH_CHECK(kv_heads > 0 && wide.dim() == 2 && wide.size(0) == T && wide.size(1) == out.size(1) * kv_heads, "mix_heads: shapes");
  check(rb_mix_heads(wide.data_ptr(), mix.data_ptr(), out.data_ptr(), (int)T, (int)H, (int)kv_heads, (int)(out.size(1) / H), is_fp32(wide), cur_stream()),
        "rb_mix_heads");
}
inline void check_segments(const torch::Tensor& slot, const torch::Tensor& ctx, const c10::optional<torch::Tensor>& cu, int64_t rows, const char* what) {
  TORCH_CHECK(is_i32(slot) && is_i32(ctx) && slot.numel() == ctx.numel(), what, ": segments");
  TORCH_CHECK(cu.has_value() ? (is_i32(*cu) && cu->numel() == slot.numel() + 1) : slot.numel() == rows, what, ": segment bounds");
}
inline int64_t check_spans(const c10::optional<torch::Tensor>& spans, const c10::optional<torch::Tensor>& first, int64_t segs, const char* what) {
  if (!spans.has_value()) return 0;
  TORCH_CHECK(is_i32(*spans) && spans->dim() == 2 && spans->size(1) == 2 && first.has_value() && is_i32(*first) && first->numel() == segs + 1, what, ": spans");
  return spans->size(0);
}
void conv_inputs(torch::Tensor qkv, c10::optional<torch::Tensor> bias, c10::optional<torch::Tensor> taps, c10::optional<torch::Tensor> state,
                 c10::optional<torch::Tensor> q_w, c10::optional<torch::Tensor> k_w, c10::optional<torch::Tensor> table, torch::Tensor q,
                 c10::optional<torch::Tensor> k_pool, c10::optional<torch::Tensor> v_pool, torch::Tensor slots, torch::Tensor ctx, torch::Tensor state_slot,
                 c10::optional<torch::Tensor> cu, c10::optional<torch::Tensor> seg_of, c10::optional<torch::Tensor> pos, int64_t kv_heads, int64_t dim,
                 int64_t vdim, int64_t rot, double eps) {
  const c10::cuda::CUDAGuard guard(qkv.device());
  check_same(qkv, q, "conv_inputs");
  const int64_t T = qkv.size(0), C = q.size(1) * dim + (k_pool.has_value() ? kv_heads * (dim + vdim) : 0);
  TORCH_CHECK(qkv.dim() == 2 && qkv.stride(1) == 1 && qkv.size(1) >= C && q.dim() == 3 && q.is_contiguous() && q.size(0) == T && k_pool.has_value() == v_pool.has_value());
  TORCH_CHECK(rot == 0 || (table.has_value() && table->scalar_type() == at::kFloat && table->is_contiguous() && table->numel() == T * rot));
  TORCH_CHECK(slots.scalar_type() == at::kLong && slots.is_contiguous() && slots.numel() == T);
  check_segments(state_slot, ctx, cu, T, "conv_inputs");
  TORCH_CHECK(!cu.has_value() || (seg_of.has_value() && is_i32(*seg_of) && seg_of->numel() == T && pos.has_value() && is_i32(*pos) && pos->numel() == T));
  const int64_t n = taps.has_value() ? taps->size(1) : 1;
  for (const auto& o : {bias, taps, q_w, k_w, state})
    if (o.has_value()) {
      check_same(qkv, *o, "conv_inputs");
      TORCH_CHECK(o->is_contiguous());
    }
  TORCH_CHECK((!bias.has_value() || bias->numel() >= C) && (!taps.has_value() || (taps->dim() == 2 && taps->size(0) >= C)), "conv_inputs: weights");
  TORCH_CHECK(n == 1 || (state.has_value() && state->dim() == 3 && state->size(1) == n - 1 && state->size(2) == C), "conv_inputs: state");
  TORCH_CHECK((!q_w.has_value() || q_w->numel() >= dim) && (!k_w.has_value() || k_w->numel() >= dim), "conv_inputs: norms");
  if (k_pool.has_value()) {
    check_same(qkv, *k_pool, "conv_inputs");
    check_same(qkv, *v_pool, "conv_inputs");
    TORCH_CHECK(k_pool->dim() == 3 && v_pool->dim() == 3 && k_pool->is_contiguous() && v_pool->is_contiguous() && k_pool->size(0) == v_pool->size(0));
    TORCH_CHECK(k_pool->size(1) == kv_heads && v_pool->size(1) == kv_heads && k_pool->size(2) == q.size(2), "conv_inputs: pools");
  }
  check(rb_conv_inputs(qkv.data_ptr(), (int)qkv.stride(0), optptr(bias), optptr(taps), (int)n, state.has_value() ? state->data_ptr() : nullptr, optptr(q_w),
                       optptr(k_w), rot ? table->data_ptr<float>() : nullptr, q.data_ptr(), k_pool.has_value() ? k_pool->data_ptr() : nullptr,
                       v_pool.has_value() ? v_pool->data_ptr() : nullptr, (const long long*)slots.data_ptr<int64_t>(), ctx.data_ptr<int>(),
                       state_slot.data_ptr<int>(), optint(cu), cu.has_value() ? optint(seg_of) : nullptr, cu.has_value() ? optint(pos) : nullptr,
                       k_pool.has_value() ? k_pool->size(0) : 0, (int)T, (int)ctx.numel(), (int)q.size(1), (int)kv_heads, (int)dim, (int)vdim, (int)q.size(2),
                       v_pool.has_value() ? (int)v_pool->size(2) : 0, (int)rot, (float)eps, is_fp32(qkv), cur_stream()),
        "rb_conv_inputs");
}
void mingru(torch::Tensor rows, torch::Tensor z_b, torch::Tensor x_b, torch::Tensor state, torch::Tensor slot, torch::Tensor ctx, c10::optional<torch::Tensor> cu,
            torch::Tensor out, int64_t width) {
  const c10::cuda::CUDAGuard guard(rows.device());
  const int64_t pitch = (width + 7) / 8 * 8, T = rows.size(0);
  for (const auto& t : {z_b, x_b, out}) {
    check_same(rows, t, "mingru");
    TORCH_CHECK(t.is_contiguous());
  }
  TORCH_CHECK(rows.dim() == 2 && rows.stride(1) == 1 && rows.size(1) >= 3 * pitch && out.dim() == 2 && out.size(0) == T && out.size(1) == pitch && z_b.numel() >= pitch &&
              x_b.numel() >= pitch && reinterpret_cast<uintptr_t>(rows.data_ptr()) % 8 == 0, "mingru: rows");
  TORCH_CHECK(state.scalar_type() == at::kFloat && state.is_contiguous() && state.dim() >= 2, "mingru: state");
  check_segments(slot, ctx, cu, T, "mingru");
  check(rb_mingru(rows.data_ptr(), z_b.data_ptr(), x_b.data_ptr(), state.data_ptr<float>(), slot.data_ptr<int>(), ctx.data_ptr<int>(), optint(cu),
                  out.data_ptr(), (int)slot.numel(), (int)width, (int)rows.stride(0), (int)state.stride(0), is_fp32(rows), cur_stream()),
        "rb_mingru");
}
// o_raw: scratch of the CUDA-core scan; without it segments run on the tensor cores.  Returns false for shapes those do not take.
bool gla(torch::Tensor rows, torch::Tensor z, torch::Tensor z_bias, torch::Tensor norm_w, torch::Tensor state, torch::Tensor slot, torch::Tensor ctx,
         c10::optional<torch::Tensor> cu, c10::optional<torch::Tensor> o_raw, c10::optional<torch::Tensor> spans, c10::optional<torch::Tensor> first,
         c10::optional<torch::Tensor> span_state, c10::optional<torch::Tensor> span_gate, torch::Tensor out, int64_t dim, int64_t vdim, int64_t gate_col,
         double eps, double root) {
  const c10::cuda::CUDAGuard guard(rows.device());
  for (const auto& t : {z_bias, norm_w, out}) {
    check_same(rows, t, "gla");
    TORCH_CHECK(t.is_contiguous());
  }
  const int64_t H = state.size(1), T = rows.size(0), segs = slot.numel();
  TORCH_CHECK(state.dim() == 4 && state.scalar_type() == at::kFloat && state.is_contiguous() && state.size(2) == dim, "gla: state");
  TORCH_CHECK(rows.dim() == 2 && rows.stride(1) == 1 && rows.size(1) >= gate_col + H * vdim && gate_col >= H * (2 * dim + vdim) && out.size(0) == T, "gla: rows");
  TORCH_CHECK(z.dim() == 2 && z.scalar_type() == at::kFloat && z.stride(1) == 1 && z.size(0) == T && z.size(1) >= H * dim, "gla: decay");
  TORCH_CHECK(z_bias.numel() == H * dim && norm_w.numel() == vdim && root > 0, "gla: weights");
  check_segments(slot, ctx, cu, T, "gla");
  const float q_scale = 1.f / std::sqrt((float)dim), inv_root = (float)(1.0 / root);
  if (cu.has_value() && !o_raw.has_value()) {
    TORCH_CHECK(rows.scalar_type() == at::kBFloat16, "gla: the 32-bit scan needs its scratch");
    const int64_t n = check_spans(spans, first, segs, "gla");
    if (n) {
      TORCH_CHECK(span_state.has_value() && span_state->scalar_type() == at::kFloat && span_state->numel() >= n * state.stride(0));
      TORCH_CHECK(span_gate.has_value() && span_gate->scalar_type() == at::kFloat && span_gate->numel() >= n * H * dim);
    }
    const int rc = rb_gla_chunk(rows.data_ptr(), z.data_ptr<float>(), (int)z.stride(0), z_bias.data_ptr(), norm_w.data_ptr(), state.data_ptr<float>(),
                                slot.data_ptr<int>(), ctx.data_ptr<int>(), cu->data_ptr<int>(), n ? spans->data_ptr<int>() : nullptr,
                                n ? first->data_ptr<int>() : nullptr, n ? span_state->data_ptr<float>() : nullptr, n ? span_gate->data_ptr<float>() : nullptr,
                                out.data_ptr(), (int)T, (int)segs, (int)n, (int)H, (int)dim, (int)vdim, (int)state.size(3), (int)rows.stride(0),
                                (int)out.size(1), (int)gate_col, (float)eps, q_scale, inv_root, cur_stream());
    if (rc == -20) return false;
    check(rc, "rb_gla_chunk");
    return true;
  }
  TORCH_CHECK(!cu.has_value() || (o_raw->scalar_type() == at::kFloat && o_raw->numel() >= T * H * vdim), "gla: scratch");
  check(rb_gla(rows.data_ptr(), z.data_ptr<float>(), (int)z.stride(0), z_bias.data_ptr(), norm_w.data_ptr(), state.data_ptr<float>(), slot.data_ptr<int>(),
               ctx.data_ptr<int>(), optint(cu), o_raw.has_value() ? o_raw->data_ptr<float>() : nullptr, out.data_ptr(), (int)T, (int)segs, (int)H, (int)dim,
               (int)vdim, (int)state.size(3), (int)rows.stride(0), (int)out.size(1), (int)gate_col, (float)eps, q_scale, inv_root, is_fp32(rows), cur_stream()),
        "rb_gla");
  return true;
}
// y: none, one or two sublayer outputs; yw: weights of their norms or none; norms: one or two weights, or none (h[0] is a copy of the stream)
void stream_step(torch::Tensor res, std::vector<torch::Tensor> y, std::vector<torch::Tensor> yw, c10::optional<torch::Tensor> ex,
                 c10::optional<torch::Tensor> expert, c10::optional<torch::Tensor> place, c10::optional<torch::Tensor> offset,
                 c10::optional<torch::Tensor> weight, std::vector<torch::Tensor> norms, std::vector<torch::Tensor> h, c10::optional<torch::Tensor> mu,
                 c10::optional<torch::Tensor> state, c10::optional<torch::Tensor> slot, c10::optional<torch::Tensor> ctx, int64_t width, double eps) {
  const c10::cuda::CUDAGuard guard(res.device());
  const int64_t T = res.size(0), pitch = res.size(1);
  TORCH_CHECK(res.dim() == 2 && res.is_contiguous() && res.scalar_type() == at::kFloat && y.size() <= 2 && (yw.empty() || yw.size() == y.size()) &&
              norms.size() <= 2 && h.size() == (norms.empty() ? 1 : norms.size()), "stream_step: operands");
  for (const auto& t : h) {
    check_same(h[0], t, "stream_step");
    TORCH_CHECK(t.is_contiguous() && t.sizes() == res.sizes());
  }
  for (const auto& t : y) {
    check_same(h[0], t, "stream_step");
    TORCH_CHECK(t.dim() == 2 && t.size(0) == T && t.stride(1) == 1 && t.size(1) >= width && reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0, "stream_step: outputs");
  }
  for (const auto* v : {&yw, &norms})
    for (const auto& t : *v) {
      check_same(h[0], t, "stream_step");
      TORCH_CHECK(t.is_contiguous() && t.numel() == pitch, "stream_step: weights");
    }
  int top = 0;
  if (ex.has_value()) {
    check_same(h[0], *ex, "stream_step");
    TORCH_CHECK(expert.has_value() && place.has_value() && offset.has_value() && weight.has_value() && is_i32(*expert) && is_i32(*place) && is_i32(*offset) &&
                weight->scalar_type() == at::kFloat && weight->is_contiguous() && expert->dim() == 2 && expert->size(0) == T && ex->is_contiguous() && ex->dim() == 2,
                "stream_step: experts");
    top = (int)expert->size(1);
  }
  if (mu.has_value()) {
    check_same(h[0], *mu, "stream_step");
    TORCH_CHECK(mu->numel() == pitch && state.has_value() && state->is_contiguous() && state->dim() == 2 && state->size(1) == pitch, "stream_step: shift");
    check_same(h[0], *state, "stream_step");
    check_segments(*slot, *ctx, c10::nullopt, T, "stream_step");
  }
  check(rb_stream_step(res.data_ptr<float>(), y.size() > 0 ? y[0].data_ptr() : nullptr, y.size() > 0 ? (int)y[0].stride(0) : 0,
                       y.size() > 1 ? y[1].data_ptr() : nullptr, y.size() > 1 ? (int)y[1].stride(0) : 0, yw.size() > 0 ? yw[0].data_ptr() : nullptr,
                       yw.size() > 1 ? yw[1].data_ptr() : nullptr, optptr(ex), ex.has_value() ? (int)ex->size(1) : 0, optint(expert), optint(place),
                       optint(offset), weight.has_value() ? weight->data_ptr<float>() : nullptr, top, norms.size() > 0 ? norms[0].data_ptr() : nullptr,
                       norms.size() > 1 ? norms[1].data_ptr() : nullptr, h[0].data_ptr(), h.size() > 1 ? h[1].data_ptr() : nullptr, optptr(mu),
                       state.has_value() ? state->data_ptr() : nullptr, optint(slot), optint(ctx), (int)T, (int)pitch, (int)width, (float)eps, is_fp32(h[0]),
                       cur_stream()),
        "rb_stream_step");
}
void token_shift(torch::Tensor n, torch::Tensor mu, torch::Tensor state, torch::Tensor out, torch::Tensor slot, torch::Tensor ctx, torch::Tensor cu,
                 torch::Tensor seg_of) {
  const c10::cuda::CUDAGuard guard(n.device());
  for (const auto& t : {mu, state, out}) {
    check_same(n, t, "token_shift");
    TORCH_CHECK(t.is_contiguous());
  }
  const int64_t T = n.size(0), pitch = n.size(1);
  TORCH_CHECK(n.is_contiguous() && n.dim() == 2 && out.sizes() == n.sizes() && mu.numel() == pitch && state.dim() == 2 && state.size(1) == pitch, "token_shift: rows");
  check_segments(slot, ctx, cu, T, "token_shift");
  TORCH_CHECK(is_i32(seg_of) && seg_of.numel() == T, "token_shift: rows");
  check(rb_token_shift(n.data_ptr(), mu.data_ptr(), state.data_ptr(), out.data_ptr(), slot.data_ptr<int>(), ctx.data_ptr<int>(), cu.data_ptr<int>(),
                       seg_of.data_ptr<int>(), (int)T, (int)pitch, is_fp32(n), cur_stream()),
        "rb_token_shift");
}
// embed [vocab][..]: a layer's own columns start at `first`
void side_gate(torch::Tensor z, torch::Tensor embed, torch::Tensor tokens, torch::Tensor out, int64_t first, int64_t dim) {
  const c10::cuda::CUDAGuard guard(z.device());
  check_same(z, embed, "side_gate");
  check_same(z, out, "side_gate");
  const int64_t T = z.size(0);
  TORCH_CHECK(z.dim() == 2 && z.stride(1) == 1 && z.size(1) >= dim && embed.dim() == 2 && embed.is_contiguous() && first >= 0 && first + dim <= embed.size(1));
  TORCH_CHECK(out.dim() == 2 && out.is_contiguous() && out.size(0) == T && out.size(1) >= dim && tokens.scalar_type() == at::kLong && tokens.is_contiguous() &&
              tokens.numel() == T, "side_gate: rows");
  const char* e = static_cast<const char*>(embed.data_ptr()) + first * embed.element_size();
  check(rb_side_gate(z.data_ptr(), (int)z.stride(0), e, embed.size(1), (const long long*)tokens.data_ptr<int64_t>(), (int)embed.size(0), out.data_ptr(), (int)T,
                     (int)dim, (int)out.size(1), is_fp32(z), cur_stream()),
        "rb_side_gate");
}
void softcap(torch::Tensor z, double cap) {
  const c10::cuda::CUDAGuard guard(z.device());
  TORCH_CHECK(z.is_contiguous() && z.scalar_type() == at::kFloat);
  check(rb_softcap(z.data_ptr<float>(), z.numel(), (float)cap, cur_stream()), "rb_softcap");
}
void moe_route(torch::Tensor logits, c10::optional<torch::Tensor> correction, torch::Tensor expert, torch::Tensor weight, torch::Tensor place, torch::Tensor row_token, torch::Tensor count,
               torch::Tensor offset, torch::Tensor tiles, torch::Tensor n_tiles, int64_t experts, int64_t outputs, int64_t groups, int64_t keep,
               int64_t group_best, int64_t tile_rows, bool renormalize, bool softmax, double weight_scale) {
  const c10::cuda::CUDAGuard guard(logits.device());
  const int64_t T = logits.size(0), top = expert.size(1);
  TORCH_CHECK(logits.dim() == 2 && logits.scalar_type() == at::kFloat && logits.stride(1) == 1 && logits.size(1) >= outputs, "moe_route: logits");
  int corr_fp32 = 0;
  if (correction.has_value()) {
    TORCH_CHECK(correction->is_contiguous() && correction->numel() >= outputs && correction->device() == logits.device(), "moe_route: correction");
    corr_fp32 = is_fp32(*correction);
  }
  TORCH_CHECK(is_i32(expert) && is_i32(place) && expert.size(0) == T && place.sizes() == expert.sizes() && weight.scalar_type() == at::kFloat &&
              weight.is_contiguous() && weight.sizes() == expert.sizes());
  TORCH_CHECK(is_i32(row_token) && row_token.numel() >= experts * T && is_i32(count) && count.numel() >= experts + 1 && is_i32(offset) &&
              offset.numel() == experts + 1 && is_i32(n_tiles) && is_i32(tiles) && tiles.dim() == 2 && tiles.size(1) == 4);
  TORCH_CHECK(tiles.size(0) >= std::min(T * top, experts) + T * top / tile_rows, "moe_route: tile list");
  check(rb_moe_route(logits.data_ptr<float>(), (int)logits.stride(0), optptr(correction), corr_fp32, expert.data_ptr<int>(), weight.data_ptr<float>(), place.data_ptr<int>(),
                     row_token.data_ptr<int>(), count.data_ptr<int>(), offset.data_ptr<int>(), tiles.data_ptr<int>(), n_tiles.data_ptr<int>(), (int)T,
                     (int)experts, (int)outputs, (int)groups, (int)keep, (int)group_best, (int)top, (int)tile_rows, (int)tiles.size(0), renormalize, softmax,
                     (float)weight_scale, cur_stream()),
        "rb_moe_route");
}
// out[sorted row] = act(x[its token, or the sorted row] * W[expert]^T); act: 0 none, 1 squared relu, 2 and 3 gated (half as many columns out)
void moe_gemm(torch::Tensor x, torch::Tensor W, torch::Tensor out, torch::Tensor tiles, torch::Tensor n_tiles, c10::optional<torch::Tensor> row_token,
              int64_t act, double limit, int64_t bn, bool full, torch::Tensor err) {
  const c10::cuda::CUDAGuard guard(x.device());
  check_same(x, W, "moe_gemm");
  check_same(x, out, "moe_gemm");
  const int64_t E = W.size(0), N = W.size(1), K = W.size(2);
  TORCH_CHECK(x.dim() == 2 && W.dim() == 3 && out.dim() == 2 && x.is_contiguous() && W.is_contiguous() && out.is_contiguous() && x.size(1) == K && out.size(1) == (act >= 2 ? N / 2 : N));
  TORCH_CHECK(is_i32(tiles) && is_i32(n_tiles) && (!row_token.has_value() || is_i32(*row_token)));
  TORCH_CHECK(row_token.has_value() ? row_token->numel() >= E * x.size(0) : x.size(0) == out.size(0), "moe_gemm: rows");
  const int cap = (int)tiles.size(0);
  if (is_fp32(x)) {
    check(rb_moe_simt(x.data_ptr(), W.data_ptr(), out.data_ptr(), tiles.data_ptr<int>(), n_tiles.data_ptr<int>(), optint(row_token), (int)x.size(0), cap,
                      (int)N, (int)K, (int)act, (float)limit, 1, cur_stream()),
          "rb_moe_simt");
    return;
  }
  check(rb_moe_gemm(x.data_ptr(), W.data_ptr(), out.data_ptr(), tiles.data_ptr<int>(), n_tiles.data_ptr<int>(), optint(row_token), (int)x.size(0),
                    (int)x.size(0), cap, (int)E, (int)N, (int)K, (int)act, (float)limit, (int)bn, full, err.data_ptr<int>(), cur_stream()),
        "rb_moe_gemm");
}
void relu2(torch::Tensor x) {
  const c10::cuda::CUDAGuard guard(x.device());
  TORCH_CHECK(x.is_contiguous());
  check(rb_relu2(x.data_ptr(), x.numel(), is_fp32(x), cur_stream()), "rb_relu2");
}
}  // namespace

void register_serving(pybind11::module_& m) {
  m.def("launch_count", []() { return (int64_t)rb_launch_count(); });
  m.def("reset_launch_count", []() { rb_reset_launch_count(); });
  m.def("gemm", &gemm);
  m.def("gemm_pair", &gemm_pair);
  m.def("fa_fwd", &fa_fwd);
  m.def("sample_v2", &sample_v2);
  m.def("decode_advance", &decode_advance);
  m.def("decode_gemm", &decode_gemm);
  m.def("gemm_splitk_plan", &gemm_splitk_plan);
  m.def("gemm_splitk", &gemm_splitk);
  m.def("embed_rows", &embed_rows);
  m.def("norm_add", &norm_add);
  m.def("hgrn2", &hgrn2);
  m.def("latent_write", &latent_write);
  m.def("latent_attn", &latent_attn);
  m.def("latent_attn_tc", &latent_attn_tc);
  m.def("head_gemm", &head_gemm);
  m.def("gate_outputs", &gate_outputs);
  m.def("glu", &glu);
  m.def("simt_gemm", &simt_gemm);
  m.def("embed_norm", &embed_norm);
  m.def("norm_add_experts", &norm_add_experts);
  m.def("sum_norm", &sum_norm);
  m.def("rope_table", &rope_table);
  m.def("projection_inputs", &projection_inputs);
  m.def("attention_inputs", &attention_inputs);
  m.def("gqa_attn", &gqa_attn);
  m.def("paged_flash", &paged_flash);
  m.def("dense_flash", &dense_flash);
  m.def("paged_decode", &paged_decode);
  m.def("talk_decode_plan", &talk_decode_plan);
  m.def("talk_decode", &talk_decode);
  m.def("talk_flash", &talk_flash);
  m.def("mix_heads", &mix_heads);
  m.def("conv_inputs", &conv_inputs);
  m.def("mingru", &mingru);
  m.def("gla", &gla);
  m.def("stream_step", &stream_step);
  m.def("token_shift", &token_shift);
  m.def("side_gate", &side_gate);
  m.def("softcap", &softcap);
  m.def("moe_route", &moe_route);
  m.def("moe_gemm", &moe_gemm);
  m.def("relu2", &relu2);
}
