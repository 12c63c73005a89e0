// C ABI of librpeg_kernels.so (sm_100a). Every function enqueues work on `stream` (a cudaStream_t
// passed as void*) and returns 0 on success or a negative argument/launch error code; nothing here
// synchronises the device. Kernels that wait on barriers take an `int status[4]` device word
// {code, where, block, extra} that stays 0 unless a bounded wait ran out.
#pragma once
#include <stdint.h>

#define RPEG_MAX_PEERS 8
#define RPEG_KV_PAGE 64

#ifdef __cplusplus
extern "C" {
#endif

// ---- gemm.cu
int rpeg_gemm_bf16(const void* A, const void* B, void* C, int M, int N, int K, int lda, int ldb, int ldc,
                   int transA, int transB, int out_fp32, int accumulate, int bn_hint, float* workspace,
                   long long workspace_elems, int* status, void* stream);
// Same GEMM, but no operand is read before gate_flags[0..gate_words) all reached min_version (bounded wait).
int rpeg_gemm_bf16_gated(const void* A, const void* B, void* C, int M, int N, int K, int lda, int ldb, int ldc,
                         int transA, int transB, int out_fp32, int accumulate, int bn_hint, float* workspace,
                         long long workspace_elems, const unsigned* gate_flags, int gate_words, unsigned min_version,
                         unsigned long long timeout_ns, int* status, void* stream);

// ---- norm_rope.cu
int rpeg_rmsnorm_fwd(const void* x, const void* res, const void* w, void* h_out, void* y, float* rstd, int T,
                     int d, float eps, void* stream);
int rpeg_rmsnorm_bwd(const void* dy, const void* x, const void* w, const float* rstd, const void* dres_in,
                     void* dx, float* dw, int T, int d, void* stream);
int rpeg_headnorm_fwd(void* buf, int ld, int col0, int nheads, int hd, const void* w, float* rstd, int T, float eps,
                      void* stream);
int rpeg_headnorm_bwd(void* dbuf, int ldd, const void* x, int ldx, int col0, int nheads, int hd, const void* w,
                      const float* rstd, float* dw, int T, void* stream);
// consumers of split-K partials: parts is fp32 [splits][rows][width], `stride` elements between splits
int rpeg_gemm_bf16_partials(const void* A, const void* B, int M, int N, int K, int lda, int ldb, float* workspace,
                            long long workspace_elems, int* k_splits_out, int* status, void* stream);
int rpeg_rmsnorm_fwd_partials(const float* parts, int splits, long long stride, const void* res, const void* w, void* h_out,
                              void* y, int T, int d, float eps, void* stream);
int rpeg_swiglu_fwd_partials(const float* parts, int splits, long long stride, void* out, long long T, int f, void* stream);
int rpeg_rope_kv_append_partials(const float* parts, int splits, long long stride, void* qkv, int ld, int q_col0, int k_col0,
                                 int v_col0, const int* seq_id, const int* pos, const float* cos_t, const float* sin_t,
                                 const int* page_table, int max_pages, void* kcache, void* vcache, int T, int H, int Hkv,
                                 int hd, void* stream);
int rpeg_rope(void* buf, const int* pos, const float* cos_t, const float* sin_t, int T, int ld, int col0,
              int nheads, int hd, int backward, void* stream);
int rpeg_swiglu_fwd(const void* gu, void* out, long long T, int f, void* stream);
int rpeg_swiglu_bwd(const void* gu, const void* dout, void* dgu, long long T, int f, void* stream);
int rpeg_add_bf16(const void* a, const void* b, void* out, long long n, void* stream);
int rpeg_embed_fwd(const int* ids, const void* table, void* out, int T, int d, void* stream);
int rpeg_embed_bwd(const int* ids, const void* dout, float* dtable, int T, int d, void* stream);

// ---- loss.cu
int rpeg_token_logprob_fwd(const void* logits, const int* targets, float* logp, float* lse, int T, int V,
                           int ld, float temperature, void* stream);
int rpeg_token_logprob_bwd(void* logits, const int* targets, const float* lse, const float* coef, int T,
                           int V, int ld, float temperature, void* stream);
int rpeg_token_entropy(const void* logits, const float* lse, float* ent, int T, int V, int ld, float temperature,
                       void* stream);
int rpeg_token_logprob_entropy_bwd(void* logits, const int* targets, const float* lse, const float* coef,
                                   const float* ent, const float* ecoef, int T, int V, int ld, float temperature,
                                   void* stream);
int rpeg_policy_loss(const float* lp, const float* old_lp, const float* ref_lp, const float* adv,
                     const float* mask, float* coef, float* acc, long long n, float clip_eps, float kl_coef,
                     float inv_denom, void* stream);
int rpeg_masked_rowsum(const float* x, const float* mask, float* out, int B, int T, void* stream);
int rpeg_dpo_loss(const float* pi_seq, const float* ref_seq, float* seq_coef, float* acc, int P, float beta,
                  void* stream);
int rpeg_expand_seq_coef(const float* seq_coef, const float* mask, float* coef, int B, int T, void* stream);
int rpeg_value_loss(const float* v, const float* ret, const float* mask, float* dv, float* acc, long long n,
                    float inv_denom, void* stream);
int rpeg_gae(const float* old_lp, const float* ref_lp, const float* values, const float* mask,
             const float* scores, float* adv, float* ret, int B, int T, float beta, float gamma, float lambda,
             int whiten, void* stream);
int rpeg_group_advantage(const float* rewards, float* out, int G, int K, void* stream);
int rpeg_sample(const void* logits, int B, int V, int ld, float temperature, int greedy,
                unsigned long long seed, const unsigned long long* seed_offset, const int* forced, int* token_out,
                float* logp_out, void* stream);
int rpeg_sample_filtered(const void* logits, int B, int V, int ld, float temperature, int top_k, float top_p,
                         unsigned long long seed, const unsigned long long* seed_offset, const int* forced, int* token_out,
                         float* logp_out, void* stream);
int rpeg_sample_f32(const void* logits, int B, int V, int ld, float temperature, int greedy, unsigned long long seed,
                    const unsigned long long* seed_offset, const int* forced, int* token_out, float* logp_out, void* stream);
int rpeg_sample_filtered_f32(const void* logits, int B, int V, int ld, float temperature, int top_k, float top_p,
                             unsigned long long seed, const unsigned long long* seed_offset, const int* forced,
                             int* token_out, float* logp_out, void* stream);
int rpeg_head_gemv(const void* h, const void* w, const float* bias, float* out, int T, int d, void* stream);
int rpeg_head_gemv_bwd(const void* h, const void* w, const float* dout, void* dh, float* dw, float* db, int T,
                       int d, void* stream);

// ---- optim.cu
int rpeg_adamw(float* p32, float* m, float* v, const float* grad, void* w16, long long n, float lr, float beta1,
               float beta2, float eps, float wd, int step, float grad_scale, const float* sumsq, int n_partials,
               float max_norm, void* stream);
int rpeg_sumsq(const float* x, long long n, float* out, void* stream);
int rpeg_flag_barrier(void* const* pads, int rank, int world, int slot, unsigned epoch, const float* payload_in,
                      float* payload_out, unsigned long long timeout_ns, int* status, void* stream);
int rpeg_dp_reduce_norm(void* const* grads, int world, long long shard_off, long long shard_n, float scale,
                        float* reduced, float* sumsq, void* stream);
int rpeg_dp_adam_push(float* p32, float* m, float* v, const float* reduced, void* const* params, int world,
                      long long shard_off, long long shard_n, float lr, float beta1, float beta2, float eps,
                      float wd, int step, const float* sumsq, int n_partials, float max_norm, void* stream);
int rpeg_copy16(const void* src, void* dst, long long nbytes, void* stream);
int rpeg_scatter_rows_by_index(const void* src, long long n, long long row_bytes, const long long* global_idx,
                               long long rows_per_rank, void* const* dst, int world, void* stream);
// Version words of pushed data: release-store `version` into word `word` of every destination flag array after
// the copies queued before it; poll flags[0..n) >= min_version with a bound (result[0] = 1 reached, 0 not yet).
// Programmatic dependent launches on/off for subsequent launches (graphs keep the setting of their capture).
void rpeg_set_pdl(int on);
int rpeg_publish_version(void* const* flag_arrays, int n_dst, int word, unsigned version, void* stream);
int rpeg_wait_flags(const unsigned* flags, int n, unsigned min_version, unsigned long long timeout_ns, int* result,
                    void* stream);
int rpeg_copy2d(const void* src, long long src_pitch, void* dst, long long dst_pitch, long long rows, long long row_bytes,
                void* stream);

// ---- gemm_rs.cu: row-parallel linear = GEMM + reduce-scatter (or all-reduce) over peer memory in one launch
int rpeg_gemm_rs(const void* A, const void* B, int M, int N, int K, int lda, int ldb, void* const* stage,
                 void* const* counters, void* const* outs, int ldo, int rank, int world, unsigned epoch, int all_gather,
                 int* status, void* stream);

// ---- ag_gemm.cu: column-parallel linear = all-gather of the activation rows + GEMM in one launch
int rpeg_ag_gemm(void* const* xs, const void* W, void* Y, void* const* readys, int M, int N, int K, int ldx, int ldw, int ldy,
                 int rank, int world, unsigned epoch, int* status, void* stream);

// ---- decode_attn.cu
int rpeg_kv_append(const void* qkv, int ld, int k_col0, int v_col0, const int* seq_id, const int* pos,
                   const int* page_table, int max_pages, void* kcache, void* vcache, int T, int Hkv, int hd,
                   void* stream);
int rpeg_rope_kv_append(void* qkv, int ld, int q_col0, int k_col0, int v_col0, const int* seq_id, const int* pos,
                        const float* cos_t, const float* sin_t, const int* page_table, int max_pages, void* kcache,
                        void* vcache, int T, int H, int Hkv, int hd, void* stream);
long long rpeg_decode_attn_scratch_bytes(int B, int H, int nsplit);
int rpeg_paged_decode_attn(const void* q, int ldq, int q_col0, const void* kcache, const void* vcache,
                           const int* page_table, int max_pages, const int* seq_lens, void* out, float* scratch,
                           int B, int H, int Hkv, int hd, int nsplit, float scale, void* stream);
// Same, for batches whose rows share their first keys in groups (page-table aliasing): group_rows [B, 8], group_shared [B],
// row_key0 [B]; scratch sized for nsplit + 1 partials.
int rpeg_paged_decode_attn_grouped(const void* q, int ldq, int q_col0, const void* kcache, const void* vcache,
                                   const int* page_table, int max_pages, const int* seq_lens, void* out, float* scratch,
                                   int B, int H, int Hkv, int hd, int nsplit, float scale, const int* group_rows,
                                   const int* group_shared, const int* row_key0, void* stream);

// ---- symm.cu
int rpeg_symm_alloc(unsigned long long bytes, void** out);
int rpeg_symm_free(void* p);
int rpeg_ipc_export(void* p, void* handle64);
int rpeg_ipc_open(const void* handle64, void** out);
int rpeg_ipc_close(void* p);
int rpeg_memset_async(void* p, int value, unsigned long long bytes, void* stream);

// ---- generate.cu
int rpeg_decode_prepare(const int* active, const int* gen_count, const int* forced_len, int* forced, int n_slots,
                        int eos, void* stream);
int rpeg_decode_advance(const int* sampled, const float* sampled_lp, int* token, int* pos, int* seq_len,
                        int* active, int* gen_count, int* out_tok, float* out_lp, int n_slots, int max_new,
                        int eos, int* n_finished, unsigned long long* step_counter, void* stream);
int rpeg_gather_rows(const void* x, const int* rows, void* out, int n, int d, void* stream);
int rpeg_scatter_rows(void* x, const int* rows, const void* src, int n, int d, int overwrite, void* stream);
int rpeg_splitk_reduce(const float* part, void* out, int M, int N, int ldc, int splits, void* stream);

// ---- flash_attn.cu
int rpeg_flash_attn_fwd(const void* qkv, int ld, int q_col0, int k_col0, int v_col0, const int* cu_seqlens,
                        int B, int max_seqlen, int T, int H, int Hkv, int hd, float scale, void* out, float* lse,
                        int* status, void* stream);

int rpeg_flash_attn_bwd(const void* qkv, int ld, int q_col0, int k_col0, int v_col0, const void* out,
                        const void* dout, const float* lse, const int* cu_seqlens, int B, int max_seqlen, int T,
                        int H, int Hkv, int hd, float scale, float* dvec, float* dq_acc, void* dqkv, int ld_dqkv,
                        int* status, void* stream);

// ---- residual_norm.cu: norms around an fp32 residual stream (`kind`: 0 activation, 1 split-K partials, 2 expert outputs,
// 3 embedding rows, 4 the stream itself); activations and weights are bf16, or fp32 with f32 = 1
int rpeg_residual_norm(int kind, const void* src, int splits, long long stride, int ld, const int* idx, const float* wts,
                       int top, int n_shared, long long shared_row0, const void* w, const void* w2, float* x, void* y,
                       int rows, int d, int dp, float eps, float w_add, int add, int f32, void* stream);

// ---- window_attn.cu / window_prefill.cu: chunked attention with a sink over the paged cache
int rpeg_rotary_append(const void* src, int splits, long long stride, int ld, int q_col0, int k_col0, int v_col0, const int* slot,
                       const int* pos, const float* cos_t, const float* sin_t, const int* page_table, int max_pages, void* q_out,
                       int ldq, void* kcache, void* vcache, int rows, int H, int Hkv, int dim, int dp, int rot_dims, int do_norm,
                       float eps, int f32, void* stream);
long long rpeg_rows_attn_scratch(int rows, int H, int dp, int nsplit);
int rpeg_rows_attn(const void* q, int ldq, const void* kcache, const void* vcache, const int* page_table, int max_pages,
                   const int* slot, const int* pos, const int* lens, const float* sink, void* out, int ldo, float* scratch,
                   int* arrive, int rows, int H, int Hkv, int dp, int window, int nsplit, float scale, int f32, int* status,
                   void* stream);
int rpeg_window_prefill(const void* q, int ldq, const void* kcache, const void* vcache, long long num_pages, const int* page_table,
                        int max_pages, const int* cu, const int* pos, const int* slot, const float* sink, void* out, int ldo, int T,
                        int B, int max_len, int H, int Hkv, int dp, int window, float scale, int* status, void* stream);

// ---- moe.cu: mixture of experts (routing, dispatch, grouped GEMM over the experts' row segments)
int rpeg_moe_route(const float* logits, int splits, long long stride, int ld, int rows, int E, int n_groups, int keep, int top,
                   int renorm, int sigmoid, int* ids, float* wts, int* ticket, int* counts, void* stream);
int rpeg_moe_dispatch(const void* x, int dp, const int* ids, const int* ticket, const float* wts, const int* counts, int rows, int E,
                      int top, void* xs, int* row_of, int* seg_off, int f32, void* stream);
int rpeg_moe_gemm(const void* A, long long a_rows_total, const void* X, const void* B, void* C, const int* seg_off, int n_routed,
                  int n_shared, int seg_rows, long long choices, int N, int K, int lda, int ldx, int ldb, int ldc, int act,
                  int bn_hint, int* status, void* stream);

// ---- gemm_f32.cu: fp32 matrix products on the CUDA cores
int rpeg_gemm_f32(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldb, int ldc, void* stream);
int rpeg_moe_gemm_f32(const float* A, const float* X, const float* B, float* C, const int* seg_off, int n_routed, int n_shared,
                      int seg_rows, int N, int K, int lda, int ldb, int ldc, int act, void* stream);
int rpeg_gemm_f32_batched(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldb, int ldc, long long a_stride,
                          long long b_stride, long long c_stride, int batch, int b_kn, void* stream);

// ---- stream_update.cu: x += mixer output + feed-forward output; y = tanh(alpha x) w + b (fp32 stream, see the source for the kinds)
int rpeg_stream_update(int kind_a, const void* a, int splits_a, long long stride_a, int ld_a, const int* ids, int kind_b, const void* b,
                       int splits_b, long long stride_b, int ld_b, const int* row_of, const float* wts, int top, int n_shared,
                       long long shared_row0, const float* alpha, const void* w, const void* bias, float* x, void* y, int rows, int dp,
                       int f32, void* stream);

// ---- latent.cu: latent attention around the projections, and on the CUDA cores
int rpeg_latent_rows(const void* src, int splits, long long stride, int ld, int rows, const int* pos, const int* slot, const float* cos_t,
                     const float* sin_t, int rot, int rot_p, float eps, int nq_col0, int nq, int nq_p, const void* nq_w, void* nq_out,
                     int kv_col0, int rank, int rank_p, const void* kv_w, void* cache, const int* page_table, int max_pages, int q_col0,
                     int H, int dim_p, void* q_nope, int ld_nope, void* q_rot, int ld_rot, int hs_rot, int ff_col0, int ff_p, void* ff_out, int f32,
                     void* stream);
int rpeg_latent_gather(const void* cache, int row_bytes, const int* page_table, int max_pages, const int* slot, const int* cu, const int* off,
                       const int* lo, int B, int rows, void* out, void* stream);
int rpeg_latent_attn_rows(const void* q, const void* cache, const int* page_table, int max_pages, const int* slot, const int* pos,
                          const int* lens, const float* sink, void* out, int rows, int H, int rank_p, int W, int window, float scale, int f32,
                          void* stream);

// ---- latent_decode.cu / latent_prefill.cu: the same on the tensor cores
int rpeg_latent_decode_ctas(int rank_p, int W);
long long rpeg_latent_decode_scratch(int rows, int H, int rank_p, int nsplit);
int rpeg_latent_decode(const void* q, const void* cache, long long num_pages, const int* page_table, int max_pages, const int* slot, const int* pos,
                       const int* lens, const float* sink, void* out, float* scratch, int rows, int H, int rank_p, int W, int window, int nsplit,
                       float scale, int* status, void* stream);
int rpeg_latent_prefill_fits(int dim_p, int rot_p, int vdim_p);
int rpeg_latent_prefill(const void* q, int ldq, int hsq, const void* kv, const void* rows, long long n_rows, int W, int rank_p, const int* cu,
                        const int* pos, const int* off, const int* lo, const float* sink, void* out, int ldo, int T, int B, int max_len, int H,
                        int dim_p, int rot_p, int vdim_p, int window, float scale, int* status, void* stream);

// ---- head_gemm.cu: C[r, h, :] = A[r, h, :] * B_h
int rpeg_head_gemm(const void* A, const void* B, void* C, int M, int N, int K, int H, int lda, int hsa, int ldc, int hsc, int b_kn, int* status,
                   void* stream);

#ifdef __cplusplus
}
#endif
