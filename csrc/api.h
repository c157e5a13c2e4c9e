// C entry points of the sm_100a kernels (one launcher per op).  Every function
// returns 0 on success, a cudaError_t value or a negative argument-check code
// otherwise, launches on `stream` and allocates nothing.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

int rb_gemm(const void* A, const void* B, void* C, const void* bias, int M, int N, int K, int lda, int ldb, int ldc,
            int a_mn_major, int b_mn_major, int out_fp32, int accumulate, int is_fp16, int force_bn, int lbo_a,
            int sbo_a, int lbo_b, int sbo_b, int* err_flag, cudaStream_t stream);

int rb_gemm_pair(const void* A, const void* B, void* C, int M, int N, int K, int lda, int ldb, int ldc, int a_mn_major,
                 int b_mn_major, int out_fp32, int accumulate, int force_bn, int* err_flag, cudaStream_t stream);

int rb_rmsnorm_fwd(const void* x, const void* res, const void* w, void* y, void* r_out, int rows, int cols, float eps,
                   int dtype, cudaStream_t st);
int rb_rmsnorm_bwd_parts(int rows, int cols);
int rb_rmsnorm_bwd(const void* x, const void* w, const void* dy, void* dx, void* dw, float* scratch, int rows, int cols,
                   float eps, int dtype, cudaStream_t st);
int rb_rope(const void* x, void* y, const float* cos_t, const float* sin_t, long long tokens, int H, int D, int backward,
            int dtype, cudaStream_t st);
int rb_swiglu_fwd(const void* in, void* out, long long rows, int F, int dtype, cudaStream_t st);
int rb_swiglu_bwd(const void* in, const void* dout, void* din, long long rows, int F, int dtype, cudaStream_t st);
int rb_adam(void* p, void* master, const void* g, float* m, float* v, long long n, int step, float lr, float b1, float b2,
            float eps, float wd, float gscale, int split, int grad_fp32, cudaStream_t st);
int rb_sumsq(const void* g, long long n, float* out, int dtype, cudaStream_t st);
int rb_copy_table(const void* table, int n_desc, const int* chunk_start, int total_chunks, int chunk_rows, int elem_size,
                  cudaStream_t st);
int rb_kv_scatter(const void* k, const void* v, void* kc, void* vc, const long long* slots, int tokens, int row_elems,
                  long long k_stride, long long v_stride, int dtype, cudaStream_t st);
int rb_int4_fake_quant(const void* x, void* out, void* scale, void* zero, int M, int N, int bm, int bn, int sym, int dtype,
                       cudaStream_t st);
int rb_fp8_block_cast(const void* w, void* q, float* scale, int M, int N, int block, int ue8m0, int dtype, cudaStream_t st);
int rb_fp8_block_dequant(const void* q, const float* scale, void* out, int M, int N, int block, int dtype, cudaStream_t st);

int rb_dense_flash(const void* q, long long q_pitch, const void* k, const void* v, const int* first, const int* blocks, const void* gate, int ld_gate,
                   int head_gate, void* out, int rows, int n, int H, int dk, int dv, long long k_rows, float scale, int* err, cudaStream_t st);
int rb_sum_norm(float* res, const void* y, const void* ex, const int* expert, const int* place, const int* offset, const float* weight, int top, int
                experts, const void* w, const void* b, const void* next_w, const void* next_b, void* h, int rows, int ldy, int pitch, int width, int
                centre, float alpha, float eps, float scale, int fp32, cudaStream_t st);
int rb_projection_inputs(const void* qkv, int ld, const void* q_w, const void* k_w, const float* table, void* q, void* k_pool, void* v_pool, const
                         long long* slots, long long pool_rows, int T, int H, int G, int dim, int vdim, int dp, int vp, int rot, int halves, float
                         eps, int fp32, cudaStream_t st);
#ifdef __cplusplus
}
#endif

#ifdef TORCH_EXTENSION_NAME
#include <pybind11/pybind11.h>
void register_more(pybind11::module_& m);
void register_serving(pybind11::module_& m);
#endif

// ---- attention / decode / sampling / fused LM head (declared again for C callers)
#ifdef __cplusplus
extern "C" {
#endif
int rb_fa_fwd(const void* q, const void* k, const void* v, void* o, float* lse, const int* cu_q, const int* cu_k,
              int num_seqs, int Tq, int Tk, int Hq, int Hkv, long long q_tok, long long q_head, long long k_tok,
              long long k_head, long long v_tok, long long v_head, int causal, float scale, int max_q_blocks, int* err,
              cudaStream_t stream);
int rb_fa_bwd(const void* q, const void* k, const void* v, const void* o, const void* d_o, const float* lse, void* dq,
              void* dk, void* dv, float* delta, float* dq_acc, const int* cu_q, const int* cu_k, int num_seqs, int Tq,
              int Tk, int Hq, int Hkv, int causal, float scale, int max_kv_blocks, int* err, cudaStream_t stream);
int rb_decode_attn_splits(int B, int Hkv, int max_ctx);
int rb_decode_attn(const void* q, const void* kc, const void* vc, const int* block_tables, const int* ctx_lens, void* out,
                   float* part_o, float* part_ml, int B, int Hq, int Hkv, int block_size, int max_blocks, int max_ctx,
                   float scale, int splits, cudaStream_t st);
int rb_decode_attn_v1(const void* q, const void* kc, const void* vc, const int* block_tables, const int* ctx_lens, void* out,
                      float* part_o, float* part_ml, int B, int Hq, int Hkv, int block_size, int max_blocks, int max_ctx,
                      float scale, int splits, cudaStream_t st);
int rb_decode_attn_tc(const void* q, const void* kc, const void* vc, const int* block_tables, const int* ctx_lens, void* out,
                      float* part_o, float* part_ml, int B, int Hq, int Hkv, int num_blocks, int block_size, int max_blocks,
                      int max_ctx, float scale, int splits, int* err, cudaStream_t st);
int rb_sample(const float* logits, int B, int V, int ld, const float* temperature, const long long* top_k,
              const float* top_p, const float* uniform, long long* tok, float* logp, cudaStream_t st);
int rb_topk_router(const float* logits, int T, int E, int K, int norm, float* w, long long* idx, float* probs,
                   cudaStream_t st);
int rb_sample_v2(const void* logits, int is_bf16, int B, int V, long long ld, const float* temperature,
                 const long long* top_k, const float* top_p, const float* uniform, long long* tok, float* logp,
                 cudaStream_t st);
int rb_decode_advance(const long long* tok_new, const float* lp_new, long long* tok_in, long long* pos, int* ctx,
                      long long* slot, const int* block_table, int max_blocks, int block_size, int* active, int* remain,
                      const long long* eos, const long long* stop_ids, int n_stop, long long* out_tok, float* out_lp,
                      int* counter, int window, const float* u_all, float* u_next, int B, cudaStream_t st);
int rb_gemm_splitk_plan(int M, int N, int K, int* bn_out);
int rb_gemm_splitk(const void* A, const void* B, void* C, const void* bias, const void* residual, float* workspace, int M,
                   int N, int K, int lda, int ldb, int ldc, int splits, int bn, int is_fp16, int* err_flag,
                   cudaStream_t stream);
int rb_gemm_ar_plan(int M, int N, int K, int* bn_out);
int rb_gemm_ar_rmsnorm(const void* A, const void* B, int M, int N, int K, int lda, int ldb, int tp, int tp_rank,
                       float* const* peer_ws, unsigned* const* peer_sig, int* state, const void* residual,
                       const void* norm_w, void* out_h, void* out_x, float eps, int splits, int bn,
                       int reduce_scatter, int b_mn_major, unsigned long long wait_ns, unsigned long long* timeline,
                       int* err_flag, cudaStream_t stream);
int rb_ag_gemm(const void* x_shard, const void* B, void* C, int M, int N, int K, int ldb, int ldc, int tp, int tp_rank,
               void* const* peer_ag, unsigned* const* peer_sig, int* state, int bn, unsigned long long wait_ns,
               int* err_flag, cudaStream_t stream);
int rb_qkv_post(const void* qkv, int ld, const void* qw, const void* kw, const float* cos_t, const float* sin_t, void* q_out,
                void* k_out, void* v_out, void* k_cache, void* v_cache, const long long* slots, int T, int nq, int nkv,
                float eps, cudaStream_t st);
int rb_splitk_swiglu(const float* ws, void* out, int M, int F, int splits, cudaStream_t st);
int rb_dp_reduce_sumsq(float* const* peer_g, unsigned* const* peer_sig, int* state, int dp, int rank, long long lo, long long n,
                       float* out, float* sumsq, float scale, unsigned long long wait_ns, int* err, cudaStream_t st);
int rb_dp_adam_allgather(void* const* peer_p, unsigned* const* peer_sig, int* state, int dp, int rank, long long lo,
                         long long n, void* master, const float* g, float* m, float* v, int step, float lr, float b1,
                         float b2, float eps, float wd, float gscale, int split, unsigned long long wait_ns, int* err,
                         cudaStream_t st);
int rb_fa_bwd_ex(const void* q, const void* k, const void* v, const void* o, const void* d_o, const float* lse, void* dq,
                 void* dk, void* dv, float* delta, float* dq_acc, const int* cu_q, const int* cu_k, int num_seqs, int Tq,
                 int Tk, int Hq, int Hkv, int causal, float scale, int max_kv_blocks, int flags, int* err,
                 cudaStream_t stream);
int rb_fa_dq_convert(const float* dq_acc, void* dq, long long n, cudaStream_t stream);
int rb_peer_barrier(unsigned* const* peer_sig, int* state, int n, int rank, int slot, int state_idx,
                    unsigned long long wait_ns, int* err, cudaStream_t st);
int rb_peer_push(const void* src, void* const* dst, int n_dst, long long nbytes, cudaStream_t st);
int rb_gemm_fp8_blockscaled(const void* A, const float* sa, const void* B, const float* sb, void* C, int M, int N, int K,
                            int lda, int ldb, int ldc, int* err, cudaStream_t stream);
int rb_grouped_gemm_fwd(const void* X, const void* W, void* Y, const int* tile_expert, int rows_cap, int N, int K, int E,
                        int* err, cudaStream_t st);
int rb_grouped_gemm_dgrad(const void* dY, const void* W, void* dX, const int* tile_expert, int rows_cap, int Nw, int Kw,
                          int E, int* err, cudaStream_t st);
int rb_grouped_gemm_wgrad(const void* dY, const void* X, void* dW, const int* expert_rows, int rows_cap, int Nw, int Kw,
                          int E, int out_fp32, int accumulate, int* err, cudaStream_t st);
int rb_decode_gemm_splits(int tiles, int k_iters);
int rb_decode_gemm(const void* x, const void* W, void* y, int Mt, int N, int K, int ldx, int ldw, int glu, int splits,
                   int* err, cudaStream_t st);
int rb_policy_loss(const float* ppo_kl, const float* adv, float* loss, float* clipfrac, float* dkl, long long n, float eps_clip,
                   float eps_clip_high, float eps_clip_c, cudaStream_t st);
int rb_lm_head_splits(int M, int N);
int rb_lm_head_logprob(const void* h, const void* W, const long long* targets, float* partials, int M, int N, int K,
                       int ldh, int ldw, int vocab_start, float inv_temp, int n_splits, int* err, cudaStream_t stream);
int rb_lm_head_dlogits(const void* h, const void* W, const long long* targets, const float* row_stats, const float* g_lp,
                       const float* g_ent, void* dlogits, int M, int N, int K, int ldh, int ldw, int ldd, int vocab_start,
                       float inv_temp, int* err, cudaStream_t stream);
// ---- composed stacks (stack_sm100.cu); fp32 = 1: 32-bit operands, 0: bf16
int rb_embed_rows(const long long* tok, const void* w, float* res, void* h, int rows, int vocab, int pitch, float scale, int fp32, cudaStream_t st);
int rb_norm_add(float* res, const void* y, const void* w, const void* next_w, void* h, int rows, int ldy, int pitch, int width,
                int groups, float eps, int fp32, cudaStream_t st);
int rb_hgrn2(const void* qfv, const void* f_bias, const void* lower, const void* norm_w, float* state, const int* slot, const int* ctx,
             const int* cu, float* o_raw, void* out, int rows, int segs, int H, int dim, int vdim, int vp, int ld, int ldo, float eps,
             int fp32, cudaStream_t st);
int rb_hgrn2_chunk(const void* qfv, const void* f_bias, const void* lower, const void* norm_w, float* state, const int* slot, const int* ctx,
                   const int* cu, const int* spans, const int* first, float* span_state, float* span_gate, void* out, int rows, int segs,
                   int n_spans, int H, int dim, int vdim, int vp, int ld, int ldo, float eps, cudaStream_t st);
int rb_gla(const void* in, const float* z, int ldz, const void* z_bias, const void* norm_w, float* state, const int* slot, const int* ctx, const int* cu,
           float* o_raw, void* out, int rows, int segs, int H, int dim, int vdim, int vp, int ld, int ldo, int gate_col, float eps, float q_scale,
           float inv_root, int fp32, cudaStream_t st);
int rb_gla_chunk(const void* in, const float* z, int ldz, const void* z_bias, const void* norm_w, float* state, const int* slot, const int* ctx,
                 const int* cu, const int* spans, const int* first, float* span_state, float* span_gate, void* out, int rows, int segs, int n_spans,
                 int H, int dim, int vdim, int vp, int ld, int ldo, int gate_col, float eps, float q_scale, float inv_root, cudaStream_t st);
int rb_mingru(const void* rows, const void* z_b, const void* x_b, float* state, const int* slot, const int* ctx, const int* cu, void* out, int segs, int
              width, int ld, int sp, int fp32, cudaStream_t st);
int rb_stream_step(float* res, const void* y0, int ldy0, const void* y1, int ldy1, const void* w0, const void* w1, const void* ex, int ldx, const int*
                   expert, const int* place, const int* offset, const float* weight, int top, const void* n0, const void* n1, void* h0, void* h1, const
                   void* mu, void* state, const int* slot, const int* ctx, int rows, int pitch, int width, float eps, int fp32, cudaStream_t st);
int rb_token_shift(const void* n, const void* mu, void* state, void* out, const int* slot, const int* ctx, const int* cu, const int* seg_of, int rows,
                   int pitch, int fp32, cudaStream_t st);
int rb_side_gate(const void* z, int ldz, const void* embed, long long lde, const long long* tok, int vocab, void* out, int rows, int dim, int pitch,
                 int fp32, cudaStream_t st);
int rb_softcap(float* z, long long n, float cap, cudaStream_t st);
int rb_conv_inputs(const void* qkv, int ld, const void* bias, const void* taps, int n, void* state, const void* q_w, const void* k_w, const float* table,
                   void* q, void* k_pool, void* v_pool, const long long* slots, const int* ctx, const int* state_slot, const int* cu, const int* seg_of,
                   const int* pos, long long pool_rows, int T, int segs, int H, int G, int dim, int vdim, int dp, int vp, int rot, float eps, int fp32,
                   cudaStream_t st);
int rb_talk_decode_plan(int H, int G, int dk, int dv, int* value_groups);
int rb_talk_decode(const void* q, const void* kc, const void* vc, const int* block_tables, const int* ctx_lens, const void* sink, const void* mix, void* out,
                   float* part_o, float* part_l, int B, int H, int G, int dk, int dv, int out_d, long long pool_rows, int page, int max_blocks, int max_ctx,
                   int window, int keep, int chunk, float scale, float cap, int splits, int* err, cudaStream_t st);
int rb_talk_flash(const void* q, const void* kc, const void* vc, const int* block_tables, const int* ctx, const int* blocks, const void* sink, void* out,
                  int rows, int n, int Hq, int Hkv, int dk, int dv, int out_d, long long pool_rows, int page, int max_blocks, int window, int keep, int
                  chunk, float scale, float cap, int* err, cudaStream_t st);
int rb_mix_heads(const void* wide, const void* mix, void* out, int rows, int H, int G, int vo, int fp32, cudaStream_t st);
int rb_latent_write(const void* raw, const void* k_rot, void* q, int ld, const void* w, void* pool, const long long* slots, const float* table, long
                    long pool_rows, int rows, int rank, int pitch, int part, int rot, int H, int dk, int dim, float eps, int fp32, cudaStream_t st);
int rb_latent_attn(const void* q, const void* pool, const int* block_tables, const int* row_seg, const int* row_pos, const int* ctx, const void* gate,
                   void* out, int rows, int H, int R, int Rv, int max_blocks, int block_size, int ld_gate, float scale, int fp32, cudaStream_t st);
int rb_latent_attn_tc(const void* q, const void* pool, const int* block_tables, const int* items, const int* ctx, const void* gate, void* out, float*
                      part_o, float* part_ml, int rows, int H, int R, int Rv, long long pool_rows, int max_blocks, int page, int n_items, int width,
                      int splits, int ld_gate, float scale, int* err, cudaStream_t st);
int rb_head_gemm(const void* x, const void* w, const void* gate, int ld_gate, void* out, int T, int H, int N, int K, long long x_tok, long long
                 x_head, int kn, int* err, cudaStream_t st);
int rb_gate_outputs(void* o, const void* gate, int ld_gate, int rows, int n, int fp32, cudaStream_t st);
int rb_glu(const void* in, void* out, long long rows, int F, int ld_in, int act, int fp32, cudaStream_t st);
int rb_simt_gemm(const void* A, const void* B, void* C, int M, int N, int K, int lda, int ldb, int ldc, int b_kn, int batch, long long sa,
                 long long sb, long long sc, int fp32, cudaStream_t st);
int rb_norm_add_experts(float* res, const void* y, const void* ex, const int* expert, const int* place, const int* offset, const float* weight, int
                        top, int experts, const void* w, const void* next_w, void* h, int rows, int ldy, int pitch, int width, int groups, float eps,
                        int fp32, cudaStream_t st);
int rb_embed_norm(const long long* tok, const void* table, const void* w, float* res, void* h, int rows, int vocab, int pitch, int width, int groups,
                  float eps, int fp32, cudaStream_t st);
int rb_rope_table(const int* pos, int offset, const double* freq, float* out, int rows, int half, cudaStream_t st);
int rb_attention_inputs(const void* qkv, int ld, const float* table, void* q, void* k_pool, void* v_pool, const long long* slots, long long pool_rows,
                        int T, int H, int G, int dim, int vdim, int dp, int vp, int rot, float eps, int fp32, cudaStream_t st);
int rb_gqa_attn(const void* q, const void* k_pool, const void* v_pool, const int* block_tables, const int* row_seg, const int* row_pos, const int*
                ctx, const void* sink, const void* gate, int ld_gate, void* out, int rows, int H, int G, int dp, int vp, int vo, int max_blocks, int
                block_size, int window, int keep, int chunk, int wide, float scale, float cap, int fp32, cudaStream_t st);
int rb_paged_flash(const void* q, const void* kc, const void* vc, const int* block_tables, const int* ctx, const int* blocks, const void* sink, const
                   void* gate, int ld_gate, void* out, int rows, int n, int Hq, int Hkv, int dk, int dv, int out_d, long long pool_rows, int page, int
                   max_blocks, int window, int keep, int chunk, int wide, float scale, float cap, int* err, cudaStream_t st);
int rb_paged_decode_tc(const void* q, const void* kc, const void* vc, const int* block_tables, const int* ctx_lens, const void* sink, const void*
                       gate, int ld_gate, void* out, float* part_o, float* part_ml, int B, int Hq, int Hkv, int dk, int dv, int out_d, long long
                       pool_rows, int page, int max_blocks, int max_ctx, int window, int keep, int chunk, float scale, float cap, int splits, int* err,
                       cudaStream_t st);
int rb_moe_route(const float* logits, int ld, const void* correction, int corr_fp32, int* expert, float* weight, int* place, int* row_token, int*
                 count, int* offset, int* tiles, int* n_tiles, int T, int E, int N, int groups, int keep, int group_best, int top, int tile_rows, int
                 cap, int renormalize, int softmax, float weight_scale, cudaStream_t st);
int rb_relu2(void* x, long long n, int fp32, cudaStream_t st);
int rb_moe_simt(const void* A, const void* B, void* C, const int* tiles, const int* n_tiles, const int* row_token, int capacity, int cap, int N, int
                K, int act, float limit, int fp32, cudaStream_t st);
int rb_moe_gemm(const void* X, const void* W, void* out, const int* tiles, const int* n_tiles, const int* row_token, int x_rows, int capacity, int
                cap, int E, int N, int K, int act, float limit, int bn, int full, int* err, cudaStream_t st);
#ifdef __cplusplus
}
#endif
