// C entry points of the kernels (raw pointers + stream); the torch bindings and C callers use these.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

// ---- counter.cpp ----
void mb_count_launch(int n);
long long mb_launch_count();
int mb_pdl_enabled(void);      // programmatic dependent launch for the kernels that support it (pdl.cuh); MILES_PDL=0 disables
void mb_set_pdl(int on);

// ---- gemm.cu ----
int mb_gemm_bf16(const void* A, const void* B, void* C, int M, int N, int K, long long lda, long long ldb, long long ldc,
                 int a_mn, int b_mn, int out_fp32, int accumulate, const void* bias, int force_bn, int* error_flag,
                 cudaStream_t stream);
int mb_gemm_bf16_splitk(const void* A, const void* B, void* C, int M, int N, int K, long long lda, long long ldb, long long ldc,
                        int out_fp32, int accumulate, const void* bias, int split_k, float* ws, int* counters, int* error_flag,
                        cudaStream_t stream);
int mb_gemm_bf16_grouped(const void* A, const void* B, void* C, int M_pad, int N, int K, int num_experts,
                         const int* tile_expert, int b_mn, int out_fp32, int force_bn, int* error_flag, cudaStream_t stream);
// ---- gemm_small.cu: weights on the 128-row MMA side, tokens in tiles of bt ∈ {16, 32, 64} ----
int mb_gemm_small(const void* X, const void* W, void* C, int tokens, int N, int K, long long ldx, long long ldw, long long ldc,
                  int out_fp32, const void* bias, int bt, int split_k, float* ws, int* counters, int* error_flag, cudaStream_t stream);
int mb_gemm_small_grouped(const void* X, const void* W, void* C, int rows, int N, int K, int num_experts, const int* tile_expert,
                          const int* used_rows, int bt, int* error_flag, cudaStream_t stream);
// ---- gemv.cu: ≤ 16 tokens (dense) / ≤ 8 tokens (MoE), no pipeline set-up ----
int mb_gemv(const void* x, long long ldx, const void* residual, const void* norm_w, float eps, const void* W, const void* bias, void* y, long long ldy,
            int out_fp32, void* res_out, void* xn_out, int M, int N, int K, int static_w, cudaStream_t s);
int mb_moe_gemv(const void* x, const void* w13, const void* w2, const int* topk_idx, const float* topk_w, void* act, void* out, int T, int k,
                int E, int expert_offset, int H, int F, float limit, float alpha, float shift, int ungated, cudaStream_t s);
int mb_gemm_bf16_grouped_wgrad(const void* dY, const void* X, void* dW, int M_pad, int N, int K, int num_experts,
                               const int* seg_offsets, int out_fp32, int accumulate, int force_bn, int* error_flag,
                               cudaStream_t stream);

// ---- elementwise.cu ----
int mb_rmsnorm_fwd(const void* x, const void* residual, const void* w, void* y, void* res_out, float* rstd, long long T, int H,
                   float eps, cudaStream_t s);
int mb_rmsnorm_bwd_blocks(long long T);
int mb_rmsnorm_bwd(const void* x, const void* w, const void* dy, const void* dres, const float* rstd, void* dx, float* dw_partial,
                   void* dw_out, int dw_fp32, long long T, int H, cudaStream_t s);
// RMSNorm backward that allocates nothing.  This entry point has no counterpart in the reference framework, whose
// kernels all take their workspaces from the PyTorch caching allocator; it exists for callers that cannot allocate:
// a C or C++ host without torch, code running under an allocator that is frozen or being snapshotted (the sleep /
// wake-up window in which the trainer's device memory is handed to the rollout engine), and latency-critical paths
// where an allocator call may synchronise the device.
//   * Same arguments and results as mb_rmsnorm_bwd minus `dw_partial`: the partial sums go to a fixed array in device
//     memory (592 × MB_RMSNORM_BWD_STATIC_MAX_H floats ≈ 9.7 MB, one per device, reserved when the module loads).
//   * H > MB_RMSNORM_BWD_STATIC_MAX_H returns MB_ERR_STATIC_SCRATCH_TOO_SMALL; mb_rmsnorm_bwd_static_strerror() gives text.
//   * The first call on each device looks up the array's address with cudaGetSymbolAddress; make that call before any
//     stream capture begins.  Later calls only launch the two kernels.
//   * The array is shared by all calls on a device and keeps its last contents.  Nothing needs to be zeroed: each call
//     writes every element it later reads.  Calls that overlap on one device race on it; the caller serialises them.
#define MB_RMSNORM_BWD_STATIC_MAX_H 4096
#define MB_ERR_STATIC_SCRATCH_TOO_SMALL (-2)
#define MB_ERR_STATIC_SCRATCH_SETUP (-3)
int mb_rmsnorm_bwd_static(const void* x, const void* w, const void* dy, const void* dres, const float* rstd, void* dx, void* dw_out,
                          int dw_fp32, long long T, int H, cudaStream_t s);
const char* mb_rmsnorm_bwd_static_strerror(int code);
int mb_colsum(const float* partial, void* out, int R, int C, int out_fp32, cudaStream_t s);
int mb_swiglu_fwd(const void* in, void* out, long long T, int F, const int* rows_ptr, cudaStream_t s);
int mb_swiglu_bwd(const void* in, const void* dout, void* din, long long T, int F, const int* rows_ptr, cudaStream_t s);
int mb_qk_norm_rope_fwd(const void* q, const void* k, long long q_stride, long long k_stride, const void* qw, const void* kw,
                        const int* positions, void* qo, void* ko, float* q_rstd, float* k_rstd, long long T, int Hq, int Hk, int D,
                        float theta, float eps, cudaStream_t s);
int mb_rope(const void* x, void* y, const int* positions, long long T, int H, int D, long long tok_stride, float theta, int inverse,
            cudaStream_t s);
int mb_qk_norm_rope_cache(const void* q, const void* k, const void* v, long long q_stride, long long k_stride, long long v_stride,
                          const void* qw, const void* kw, const int* positions, void* qo, void* ko, void* kc, void* vc,
                          const long long* slots, long long T, int Hq, int Hk, int D, float theta, float eps, cudaStream_t s);
int mb_qk_norm_rope_bwd_blocks(long long T, int Hn);
int mb_qk_norm_rope_bwd(const void* x, long long x_stride, const void* w, const float* rstd, const void* dy, const int* positions,
                        void* dx, long long dx_stride, float* dw_partial, void* dw_out, long long T, int Hn, int D, float theta,
                        cudaStream_t s);
int mb_kv_cache_write(const void* k, const void* v, long long k_stride, long long v_stride, void* kc, void* vc,
                      const long long* slots, long long T, int row_elems, cudaStream_t s);
int mb_adamw(float* master, const float* grad, float* m, float* v, const float* decay_mask, const float* scale_ptr, void* param_out,
             int out_bf16, long long n, float lr, float b1, float b2, float eps, float wd, int step, cudaStream_t s);

// ---- attention.cu ----
int mb_flash_fwd(const void* q, const void* k, const void* v, void* o, float* lse, const int* cu_seqlens, int batch, int max_seqlen,
                 int total_tokens, long long q_stride, long long k_stride, long long v_stride, int Hq, int Hkv, int D, float scale,
                 int causal, cudaStream_t s);
int mb_flash_bwd_tc(const void* q, const void* k, const void* v, const void* dout, const float* lse, const float* delta, void* dq,
                    void* dk, void* dv, const int* cu_seqlens, int batch, int max_seqlen, int total_tokens, long long q_stride,
                    long long k_stride, long long v_stride, int Hq, int Hkv, float scale, int causal, int* error_flag, cudaStream_t s);
int mb_attn_delta(const void* o, const void* dout, float* delta, int total_tokens, int Hq, int D, cudaStream_t s);
int mb_flash_bwd(const void* q, const void* k, const void* v, const void* o, const void* dout, const float* lse, float* delta,
                 void* dq, void* dk, void* dv, const int* cu_seqlens, int batch, int max_seqlen, int total_tokens, long long q_stride,
                 long long k_stride, long long v_stride, int Hq, int Hkv, int D, float scale, int causal, cudaStream_t s);
int mb_paged_decode(const void* q, const void* kc, const void* vc, const int* block_table, const int* seq_lens, void* out,
                    float* part_o, float* part_ml, int batch, int max_blocks, int block_size, int Hq, int Hkv, int D, float scale,
                    int num_splits, cudaStream_t s);

// ---- attention_tc.cu (tcgen05 forward, head_dim 128) ----
int mb_flash_fwd_tc(const void* q, const void* k, const void* v, void* o, float* lse, const int* cu_seqlens, int batch, int max_seqlen,
                    int total_tokens, long long q_stride, long long k_stride, long long v_stride, int Hq, int Hkv, float scale,
                    int causal, int* error_flag, const int* cu_seqlens_k, int total_k_tokens, cudaStream_t s);
int mb_flash_fwd_tc_ctas_per_sm(void);

// ---- debug.cuh: index checks of the debug build (each returns −1 in a build without them) ----
int mb_elementwise_bounds_set_limit(int which, long long value);
int mb_elementwise_bounds_read(long long* out4, int clear);
int mb_moe_bounds_set_limit(int which, long long value);
int mb_moe_bounds_read(long long* out4, int clear);
int mb_paged_bounds_set_limit(int which, long long value);
int mb_paged_bounds_read(long long* out4, int clear);

// ---- moe.cu ----
int mb_router_topk(const float* logits, float* probs, float* topk_w, int* topk_idx, long long T, int E, int K, int normalize,
                   cudaStream_t s);
int mb_moe_align(const int* idx, int n, const int* n_ptr, int E, int expert_offset, int* seg_offsets, int* tile_expert, int* row_src,
                 int* dst_row, int max_rows, cudaStream_t s);
int mb_moe_align_pad(const int* idx, int n, const int* n_ptr, int E, int expert_offset, int* seg_offsets, int* tile_expert,
                     int* row_src, int* dst_row, int max_rows, int pad, cudaStream_t s);
int mb_moe_gather(const void* x, void* x_perm, const int* row_src, const int* seg_offsets, int E, int k, int H, int max_rows,
                  cudaStream_t s);
int mb_moe_combine(const void* y_perm, const float* w, const int* dst_row, void* out, long long T, int k, int H, int identity_rows,
                   cudaStream_t s);
int mb_moe_combine_bwd(const void* dout, const void* y_perm, const float* w, const int* row_src, const int* seg_offsets, int E,
                       void* dy_perm, float* dw, int k, int H, int max_rows, cudaStream_t s);

// ---- misc.cu ----
int mb_sample_logprob_split(const float* logits, const float* temperature, const uint8_t* greedy, const long long* seeds, long long step,
                            long long* tokens, float* logprobs, int B, int V, int parts, float* ws, int* counters, cudaStream_t s);
int mb_decode_advance(const long long* o_tok, const float* o_lp, const int* o_routed, long long* h_tok, float* h_lp, int* h_routed,
                      int routed_per_row, int* tok, int* pos, int* len, const int* block_table, int max_blocks, int block_size,
                      long long* slot, long long* seed, int B, int vocab, int* error_flag, int* prev, cudaStream_t s);
int mb_sample_logprob(const float* logits, const float* temperature, const uint8_t* greedy, const long long* seeds, long long step,
                      long long* tokens, float* logprobs, int B, int V, cudaStream_t s);
int mb_logit_stats(const float* logits, long long ld, const long long* targets, float* stats, long long R, int Vc, int v0,
                   float inv_temp, int first, cudaStream_t s);
int mb_logit_stats_finish(const float* stats, float* logp, float* ent, float* lse, long long R, cudaStream_t s);
int mb_logit_grad(const float* logits, long long ld, const long long* targets, const float* lse, const float* ent, const float* g_lp,
                  const float* g_ent, void* dlogits, long long ldd, long long R, int Vc, int v0, float inv_temp, cudaStream_t s);

// ---- quant.cu ----
int mb_mxfp8_quant(const void* x, void* q, void* scales, long long numel, cudaStream_t s);
int mb_fp8_block_quant(const void* w, void* q, float* scale_inv, int M, int N, cudaStream_t s);
int mb_int4_fake_quant(const void* x, void* y, float* scales, int M, int N, int bm, int bn, int symmetric, cudaStream_t s);
int mb_block_fake_quant(const void* x, void* y, long long numel, int mode, cudaStream_t s);
int mb_nvfp4_qdq(const void* x, void* y, const float* global_amax, long long numel, int four_over_six, cudaStream_t s);
int mb_absmax(const void* x, float* out, long long numel, cudaStream_t s);

// ---- comm.cu (peer-memory kernels; *_ptrs are host arrays of `world` device addresses, one per rank) ----
int mb_barrier(const long long* flag_ptrs, int rank, int world, int channel, int* epochs, int* err, cudaStream_t s);
int mb_ar_add_rmsnorm(const long long* partial_ptrs, int world, const void* residual, const void* w, void* y, void* res_out,
                      long long T, int H, float eps, cudaStream_t s);
int mb_rs_reduce_sqnorm(const long long* grad_ptrs, int world, int rank, long long lo, long long hi, const float* norm_weight,
                        float* sqnorm, cudaStream_t s);
int mb_adam_allgather(float* master, const float* grad_shard, float* m, float* v, const float* decay_mask, const float* sqnorm,
                      float clip, const long long* param_ptrs, int world, long long lo, long long n, float lr, float b1, float b2,
                      float eps, float wd, int step, cudaStream_t s);
int mb_moe_dispatch(const void* x, const int* topk_idx, long long n_pairs, int k, int H, int e_local, int rank,
                    const long long* recv_x_ptrs, const long long* recv_meta_ptrs, const long long* counter_ptrs, int world,
                    int capacity, int* sent_row, int* err, cudaStream_t s);
int mb_moe_dispatch_signal(const void* x, const int* topk_idx, long long n_pairs, int k, int H, int e_local, int rank,
                           const long long* recv_x_ptrs, const long long* recv_meta_ptrs, const long long* counter_ptrs, int world,
                           int capacity, int* sent_row, int* err, const long long* flag_ptrs, int channel, int* epochs, int* ticket,
                           cudaStream_t s);
int mb_moe_recv_align(const void* meta, int* counter, int capacity, int E, int* seg_offsets, int* tile_expert, int* row_src, int max_rows,
                      int pad, const long long* flag_ptrs, int rank, int world, int channel, const int* epochs, int* err, cudaStream_t s);
int mb_moe_return_signal(const void* y_perm, const int* row_src, const void* meta, const int* seg_offsets, int E, int H, int max_rows,
                         const long long* ret_ptrs, int world, const long long* flag_ptrs, int rank, int channel, int* epochs, int* ticket,
                         cudaStream_t s);
int mb_moe_combine_wait(const void* ret, const float* w, const int* sent_row, void* out, long long T, int k, int H,
                        const long long* flag_ptrs, int rank, int world, int channel, const int* epochs, int* err, cudaStream_t s);
int mb_moe_scatter_known(const void* rows_in, int src_by_pair, const int* topk_idx, const int* sent_row, long long n_pairs, int k,
                         int H, int e_local, const long long* recv_x_ptrs, int world, cudaStream_t s);
int mb_moe_return(const void* y_perm, const int* row_src, const void* meta, const int* seg_offsets, int E, int H, int max_rows,
                  const long long* ret_ptrs, int world, cudaStream_t s);
int mb_recv_expert_ids(const void* meta, int* counter, int capacity, int* expert_ids, int* n_out, int clear_counter, cudaStream_t s);
int mb_sum_rows(const long long* src_ptrs, int world, void* out, long long numel, cudaStream_t s);
int mb_gather_rows(const long long* src_ptrs, int world, void* out, long long bytes_per_rank, cudaStream_t s);
int mb_stats_merge(const long long* stats_ptrs, int world, long long R, float* logp, float* ent, float* lse, cudaStream_t s);

// ---- extra.cu (other model families, quantisation tools) ----
int mb_grouped_rmsnorm(const void* x, int x_fp32, const float* w, float* out, float* rstd, long long T, int n, int C, float eps,
                       cudaStream_t s);
int mb_short_conv(const void* x, int fp32, const float* w, const int* bos, void* y, long long T, int D, int W, cudaStream_t s);
int mb_mhc_mix(const void* x, const void* res, const float* h_res, const float* h_post, void* out, int fp32, long long T, int n, int d,
               cudaStream_t s);
int mb_mhc_aggregate(const void* x, int fp32, const float* pre, float* out, long long T, int n, int d, cudaStream_t s);
int mb_hc_combine(const void* res, const void* y, const float* h_post, void* out, int fp32, long long T, int n, int C, cudaStream_t s);
int mb_act_quant_1x128(const void* x, void* q, void* qdq, float* scales, long long M, int N, int round_scale, cudaStream_t s);
int mb_fp8_dequant(const void* q, const float* scale_inv, const void* e8m0, void* out, long long M, int N, cudaStream_t s);
int mb_gather_rows_host(const void* table_dev, const long long* ids, void* out, long long n, int row_bytes, long long table_rows,
                        cudaStream_t s);

// ---- gemm_mxfp8.cu (block-scaled: e4m3 payload [rows, K] + e8m0 scales [rows, K/32]; K % 128 == 0) ----
int mb_gemm_mxfp8(const void* A, const void* sa, const void* B, const void* sb, void* C, int M, int N, int K, long long ldc,
                  int* error_flag, cudaStream_t stream);
int mb_gemm_mxfp8_grouped(const void* A, const void* sa, const void* B, const void* sb, void* C, int M_pad, int N, int K, int E,
                          const int* tile_expert, long long ldc, int* error_flag, cudaStream_t stream);

// ---- sparse_attn.cu ----
int mb_sparse_attention_fwd(const void* q, const void* k, const void* v, const int* indices, const float* sink, void* out, float* lse,
                            long long T, int H, int Hk, int D, int Dv, int K, long long Tkv, float scale, cudaStream_t s);

// ---- weight_sync.cu (one launch per bucket of tensors; dst may be peer memory) ----
int mb_multi_copy(const long long* table, const long long* prefix, int n, long long total_chunks, cudaStream_t s);
int mb_multi_copy2d(const long long* table, const long long* prefix, int n, long long total_items, int qdq, cudaStream_t s);
int mb_multi_mxfp8(const long long* table, const long long* prefix, int n, long long total_chunks, int qdq, cudaStream_t s);

// ---- mixers.cu (layer-by-layer decoders; f32: tensors of the model's dtype are float instead of bf16) ----
// xb (the copy in the model's dtype) may be null; freq [D / 2 up] (optional): sines and cosines of positions · freq are added
int mb_bigram_embedding(const int* tok, const int* prev, const void* embed, const void* table, long long buckets, long long mul_prev,
                        long long mul_cur, const int* positions, const double* freq, float* x, void* xb, int T, int D, int f32, cudaStream_t s);
// x += mult · y / rms(y) · nw · ls (ls null: 1); xb = x, or with fw x / rms(x) · fw · gain
int mb_output_norm(float* x, const void* y, const void* nw, const void* ls, float mult, const void* fw, float gain, void* xb, int T, int D,
                   float eps, int f32, cudaStream_t s);
// out = z²·softplus(act[0]) + z/2 for z > 0, (½ + softplus(act[1]))·(exp(z) − 1 − z) + z/2 else (n values)
int mb_xielu(const void* z, const void* act, void* out, long long n, int f32, cudaStream_t s);
// out[t, i] = gelu(z[t, i]) · table[tok[t], col + i] (tanh form), n columns
int mb_gelu_rows(const void* z, long long ld, const int* tok, const void* table, long long table_ld, int col, void* out, int T, int n, int f32,
                 cudaStream_t s);
// x ← cap · tanh(x / cap); exact: in double precision
int mb_softcap(float* x, long long n, float cap, int exact, cudaStream_t s);
// out = o / rms(o) · w · sigmoid(gate), every head of V channels by itself (w [V], gate [T, H·V] rows of gate_ld)
int mb_head_gated_norm(const void* o, const void* w, const void* gate, long long gate_ld, void* out, long long T, int H, int V, float eps, int f32,
                       cudaStream_t s);
// rows (optional, device): rows in use
int mb_clamped_glu(const void* in, long long ld_in, void* out, long long ld_out, long long T, int F, float limit, float alpha, float shift,
                   const int* rows, int f32, cudaStream_t s);
// x ← max(x, 0)² (n values a row, rows of them or as many as the device count says)
int mb_relu_square(void* x, long long T, int n, const int* rows, int f32, cudaStream_t s);
// out = x / rms(x) · w, each of `parts` equal parts of a row by its own root mean square
int mb_part_norm(const void* x, long long ld, const void* w, void* out, int T, int C, int parts, float eps, int f32, cudaStream_t s);
// s = x + mult·(y1·s1 + y2·s2 + s2·Σ_j weights[t, j]·rows[dst[t, j]]) + extra → to; h = rmsnorm(s)·(nw + shift)·gain (nw null: s), h2 the
// same with nw2 (every pointer but x may be null; a null scale is 1; at most one of y2 and rows where s2 is given)
typedef struct {
  const float* x;
  float* to;
  const void *y1, *y2, *rows;
  const float* weights;
  const int* dst;
  const float* extra;
  const void *s1, *s2;
  const void *nw, *nw2;
  void *h, *h2;
  int T, D, k;
  float eps, shift, gain, mult;
} MbSumNorm;
int mb_sum_norm(MbSumNorm p, int f32, cudaStream_t s);
int mb_gated_norm(const void* o, const void* w, const void* gate, long long gate_ld, void* out, int T, int C, float eps, int f32,
                  cudaStream_t s);
// gemv.cu: output norm + layer scale + fp32 residual in front of a projection of ≤ 16 rows
int mb_gemv_output_norm(const float* x, const void* y, const void* norm_w, const void* scale_w, float mult, const void* next_w, float eps,
                        const void* W, void* out, long long ldo, float* x_out, int M, int N, int K, int static_w, cudaStream_t s);
// gemv.cu: sum of an fp32 residual and up to two sublayer outputs (each times a scale vector, if given), its norm, and up to two products of
// it, for ≤ 16 rows.  x32 null: plain products of x [M, K].  W2 [N2, K] gives out2 (+ bias2), fp32 or bf16; with norm_w2 its rows are the sum
// normed by that weight.  Norm weights count from `shift`.  xn_out: the normed sum (by norm_w2 if there is one).
typedef struct {
  const float* x32;
  const void *y1, *s1, *y2, *s2;
  const float* extra;
  const void *x, *x2;                        // plain rows, ldx elements apart; x2: those of the second product (null: x)
  long long ldx;
  const void *norm_w, *norm_w2;
  float eps, shift, mult;                    // mult: factor on the addends; norm_w null: the sum as it is
  const void* W;
  void* y;
  long long ldy;
  const void *W2, *bias2;
  void* out2;
  long long ld2;
  int out2_fp32;
  float* x_out;
  void* xn_out;
  int M, N, N2, K, static_w;
} MbGemvSum;
int mb_gemv_sum_norm(MbGemvSum a, cudaStream_t s);
// ---- what attention kernels do to scores and outputs besides scale and softmax (null: nothing) ----
typedef struct {
  const void *r1, *r2;                       // [heads]: r1 · ln(1 + r2 · distance) off the scores
  const void* gate;                          // [T, heads·vdim] rows of gate_ld: outputs times its sigmoid
  long long gate_ld;
} MbScores;
// ---- paged_attend.cu ----
typedef struct {
  int heads, group, dk, dv;                  // query head h uses key head h / group
  long long q_row, q_head, k_row, k_head, v_row, v_head, o_row;   // strides in elements: token (slot) and head
  int window, keep;                          // keys a token sees (0: all), first keys that stay visible
  int chunk;                                 // tokens see their own chunk of this many positions (0: no chunks; without a window)
  float scale;
} MbAttend;
// out_f32: rows of floats whatever the dtype of the rest
int mb_paged_attend(const void* q, const void* kc, const void* vc, const int* block_table, int max_blocks, int block_size,
                    const int* token_seq, const int* positions, const long long* slots, const void* sink, void* out, int T, MbAttend A,
                    MbScores x, int f32, int out_f32, cudaStream_t s);
// ---- window_prep.cu ----
typedef struct {
  int heads, kv_heads, dim, vdim, rot, window, keep, q_pitch;   // q_pitch: elements per head of the prepared queries (zero-padded)
  int chunk;                                                    // as in MbAttend
} MbWindow;
typedef struct {                             // what reads the same projection beside the attention (null: nothing)
  const float* logits;
  float* weights;
  int* index;
  int experts, top;
  const void* glu_in;
  void* glu_out;
  long long glu_ld_in, glu_ld_out;
  int ff;
  float limit, alpha, shift;
  // grouped: choice by sigmoid scores plus `correction` (or null) among the `keep` best groups, weights from the scores times `scale`;
  // else the largest logits, weights by their softmax
  int grouped, groups, keep;
  float scale;
  const void* correction;
} MbAside;
// kc, vc null: the layer reads another's keys and values, its projection has none.  v_norm: values over their root mean square per head.
int mb_window_prep(const void* proj, long long ld, const int* positions, const long long* slots, const double* freq, float magnitude,
                   const void* q_norm, const void* k_norm, int v_norm, float eps, void* kc, void* vc, void* q, int T, MbWindow L, MbAside a,
                   int f32, cudaStream_t s);
// ---- diff_prep.cu (differential attention: two score maps per head over the same values) ----
// Query heads 2h and 2h + 1 are the maps of head h; a key head is [map 1 | map 2], a query row has zeros in the other map's half, so that
// the attention kernels see heads = 2·(query heads) of dim = 2·(map size).  What is left of a pair of outputs a1, a2:
// o = a1 − lam·a2, o / rms(o) · gain · sigmoid(gate of the head).
typedef struct {
  const float* lam;                          // device scalar; null: ordinary attention
  const void* gate;                          // [T, heads / 2] rows of gate_ld, before the sigmoid
  long long gate_ld;
  float gain, eps;
} MbDiff;
typedef struct {
  int heads, kv_heads, dim, vdim, q_pitch;   // heads, dim: of the design (one map's size); kv_heads 0: keys and values of another layer
  float eps, temp_coef;                      // queries times 1 + coef · ln(⌊(position + 1) / every⌋ + 1)
  double temp_every;
  float diff;
} MbDiffPrep;
// lvec: lq1, lk1, lq2, lk2 [4, dim]; lam ← exp(lq1·lk1) − exp(lq2·lk2) + diff
int mb_diff_prep(const void* proj, long long ld, const int* positions, const long long* slots, const void* q_norm, const void* k_norm,
                 const void* lvec, float* lam, void* kc, void* vc, void* q, int T, MbDiffPrep L, MbAside a, int f32, cudaStream_t s);
// a [T, 2·heads, vdim] floats → out [T, heads·vdim] rows of o_row
int mb_diff_combine(const float* a, void* out, long long o_row, int T, int heads, int vdim, MbDiff d, int f32, cudaStream_t s);
// ---- short_conv.cuh ----
typedef struct {
  int at, channels, taps;                    // first column of the inputs in a row of the projection
  const void *w, *b;                         // [channels, taps], [channels] (null: no bias)
  float* ring;                               // [slots, taps, channels]: the inputs of the last positions, by position mod taps (null: taps 1)
  const int* slots;                          // per sequence
  const int* positions;                      // per token
} MbConv;
// ---- delta_*.cu (gated delta rule: S ← diag(g)·S, S ← S + k (β (v − Sᵀk))ᵀ, o = Sᵀq) ----
// A row of the projection is [q: G·K | k: G·K | v: H·V | … | β: H at column beta_at]; q, k and v pass a causal convolution and silu, then q
// and k become unit vectors (q over √K on top).  g = exp(−exp(A_log)·softplus(raw + dt_bias)), raw [T, H·K] rows of raw_ld.
typedef struct {
  int H, G, K, V, taps, beta_at;
  const void* conv_w;                        // [2·G·K + H·V, taps]
  const void *A_log, *dt_bias;               // [H], [H·K]
  float* state;                              // [slots, H, K, V]
  float* ring;                               // as in MbConv
  const int* slots;
  const int* positions;
  const void* raw;
  long long raw_ld;
} MbDelta;
// Convolution of any pieces (tiles as in mb_ssm_conv): act [T, channels].
int mb_delta_conv(const void* proj, long long ld, MbDelta m, const int* tiles, const int* cu_q, int n_tiles, void* act, int f32, cudaStream_t s);
// Any pieces token by token from the convolution's outputs (cu_q null: one token per sequence); out [T, H·V] = o.
int mb_delta_seq(const void* proj, long long ld, const void* act, MbDelta m, const int* cu_q, void* out, int B, int f32, cudaStream_t s);
// One token per sequence in one launch: convolution, state, and o over its root mean square per head, times norm_w [V] and sigmoid(gate).
// Sizes: mb_delta_step_ok(K, V).
int mb_delta_step(const void* proj, long long ld, MbDelta m, const void* norm_w, const void* gate, long long gate_ld, float eps, void* out, int B,
                  int f32, cudaStream_t s);
int mb_delta_step_ok(int K, int V);
// Long pieces in chunks of 64 tokens on tensor cores (bf16; K, V multiples of 8 up to 128).  chunks [n_chunks][4]: sequence, first token,
// end; parts [n_parts][4]: first chunk, chunks, sequence (a part's chunks follow one another; a sequence has one part).  scratch:
// mb_delta_chunk_bytes(K, V) per chunk and head.  warps (2, 4 or 8): 16 value columns each that a CTA of the second kernel takes.
long long mb_delta_chunk_bytes(int K, int V);
int mb_delta_chunk(const void* proj, long long ld, const void* act, MbDelta m, const int* chunks, const int* parts, void* scratch, void* out,
                   int T, int n_chunks, int n_parts, int warps, int* error_flag, cudaStream_t s);
// ---- ssm_*.cu (state-space mixer: S ← exp(−exp(A_log)·dt)·S + dt·B xᵀ, y = Sᵀ C + D·x) ----
// A row of the projection is [z: H·V | x: H·V | B: G·N | C: G·N | dt: H]; x, B and C pass a causal convolution of `taps` columns and silu.
typedef struct {
  int H, V, N, G, taps;
  const void *conv_w, *conv_b;               // [H·V + 2·G·N, taps], [H·V + 2·G·N]
  const void *dt_bias, *A_log, *D;           // [H]
  float* state;                              // [slots, H, N, V]
  float* ring;                               // [slots, taps, channels]: the inputs of the last positions, by position mod taps (null: taps 1)
  const int* slots;                          // per sequence
  const int* positions;                      // per token
} MbSsm;
// Convolution, step sizes and log decays of any pieces.  tiles [n][4]: first token, end (at least taps − 1 tokens but for a piece's last tile),
// sequence, 1 for a piece's first tile; null: one token per sequence.  xbc [T, channels], dt and la [T, H].
int mb_ssm_conv(const void* proj, long long ld, MbSsm m, const int* tiles, const int* cu_q, int n_tiles, void* xbc, float* dt, float* la, int T,
                MbAside a, int f32, cudaStream_t s);
// One token per sequence: convolution, state, gate in one kernel; out [T, H·V] = y · silu(z).  V % 4 == 0.
int mb_ssm_step(const void* proj, long long ld, MbSsm m, void* out, int B, MbAside a, int f32, cudaStream_t s);
// Any pieces token by token (cu_q null: one token per sequence), from what mb_ssm_conv left.
int mb_ssm_seq(const void* proj, long long ld, const void* xbc, const float* dt, const float* la, MbSsm m, const int* cu_q, void* out, int B,
               int f32, cudaStream_t s);
// Long pieces in chunks on tensor cores (bf16; N, V multiples of 8 up to 128).  segs, seq_segs as in mb_linear_chunk; seg_state [n_seg, H, N, V]
// and seg_decay [n_seg, H] scratch, null when every sequence is one segment.
int mb_ssm_chunk(const void* proj, long long ld, const void* xbc, const float* dt, const float* la, MbSsm m, const int* segs, const int* seq_segs,
                 float* seg_state, float* seg_decay, void* out, int n_seq, int n_seg, cudaStream_t s);
int mb_ssm_heads_per_cta(int H, int V, int G);
// ---- window_decode.cu (bf16 tensor cores, splits joined inside a cluster) ----
int mb_window_decode(const void* q, const void* kc, const void* vc, const int* block_table, int max_blocks, int block_size, const int* token_seq,
                     const int* positions, const long long* slots, const void* sink, void* out, long long o_row, int T, float scale, int splits,
                     MbWindow L, MbDiff d, MbScores x, cudaStream_t s);
// ---- attention_window_tc.cu (tcgen05, keys and values straight from the pages) ----
int mb_window_prefill(const void* q, const void* kc, const void* vc, void* o, long long o_row, const void* sink, const int* cu_q,
                      const int* positions, const int* block_table, int max_blocks, int block_size, int num_blocks, int n_seq, int max_q,
                      int t_long, float scale, MbWindow L, MbDiff d, MbScores x, int* error_flag, cudaStream_t s);
// ---- experts_any.cu ----
// alpha 0: w13 is [E, F, H] (no gate), the activation the square of relu
int mb_experts_any(const void* x, const void* w13, const void* w2, const int* index, const float* weights, void* act, void* out, int T, int k,
                   int E, int H, int F, float limit, float alpha, float shift, int f32, cudaStream_t s);
// ---- latent_attn.cu ----
typedef struct {
  int heads, dim, rot, vdim, rank, rank_p, pitch;   // a cached row: [rank, 0 … rank_p, rot, 0 … pitch)
} MbLatent;
// q [T, heads·(dim + rot)] rows of q_ld, kv [T, rank + rot] rows of kv_ld (read with kv_norm)
int mb_latent_prep(const void* q, long long q_ld, const void* kv, long long kv_ld, const int* positions, const long long* slots, const double* freq,
                   float magnitude, const void* kv_norm, float eps, void* cache, void* q_abs, void* q_full, int T, int t_long, int q_nope,
                   int q_width, MbLatent L, int f32, cudaStream_t s);
// gate (optional): y times the sigmoid of gate[t·gate_ld + h·N + n]
int mb_head_linear(const void* x, long long x_t, long long x_h, const void* w, int w_nk, void* y, long long y_t, long long y_h, int T,
                   int H, int N, int K, const void* gate, long long gate_ld, int f32, cudaStream_t s);
int mb_latent_attend(const void* q, const void* cache, const int* block_table, int max_blocks, int block_size, const int* token_seq,
                     const int* positions, const long long* slots, const void* sink, void* out, int T, float scale, int window, MbLatent L,
                     int f32, cudaStream_t s);
// ---- latent_decode.cu (bf16 tensor cores) ----
int mb_latent_gather(const void* cache, const int* block_table, int max_blocks, int block_size, const int* cu_k, const int* base, void* out,
                     int n_seq, int total, int pitch, cudaStream_t s);
int mb_head_linear_mma(const void* x, long long x_t, long long x_h, const void* w, int w_nk, void* y, long long y_t, long long y_h, int T,
                       int H, int N, int K, const void* gate, long long gate_ld, cudaStream_t s);
int mb_latent_decode(const void* q, const void* cache, const int* block_table, int max_blocks, int block_size, const int* token_seq,
                     const int* positions, const long long* slots, const void* sink, float* part_o, float* part_ml, void* out, int T,
                     float scale, int window, int splits, int num_blocks, MbLatent L, int* error_flag, cudaStream_t s);
// ---- latent_decode_tc.cu (tcgen05; the split part of mb_latent_decode for pages of a multiple of 64 tokens) ----
int mb_latent_decode_tc(const void* q, const void* cache, const int* block_table, int max_blocks, int block_size, const int* token_seq,
                        const int* positions, const long long* slots, float* part_o, float* part_ml, int T, float scale, int window,
                        int splits, int num_blocks, MbLatent L, int* error_flag, cudaStream_t s);
// ---- attention_latent_tc.cu (tcgen05) ----
int mb_latent_prefill(const void* q, const void* kv, const void* lat, void* o, const void* sink, const void* gate, long long gate_ld, const int* cu_q,
                      const int* cu_k, int n_seq, int max_q, int t_long, int tk, float scale, int window, MbLatent L, int* error_flag,
                      cudaStream_t s);
// ---- linear_state.cu ----
int mb_linear_state(const void* proj, long long ld, const float* decay, float* state, const int* state_slots, const int* cu_q,
                    const int* positions, void* out, int B, int H, int dk, int dv, int f32, cudaStream_t s);
// ---- linear_chunk.cu (bf16 tensor cores) ----
int mb_linear_chunk(const void* proj, long long ld, const float* decay, float* state, const int* slots, const int* positions, const int* segs,
                    const int* seq_segs, float* seg_state, void* out, int n_seq, int n_seg, int H, int dk, int dv, cudaStream_t s);

// ---- gemm_comm.cu ----
int mb_ag_gemm(const long long* xg_ptrs, const void* W, void* Y, int* block_counters, int rows_per_rank, int N, int K, int rank,
               int world, const long long* flag_ptrs, int channel, int epoch, int* error_flag, cudaStream_t s);
int mb_comm_configure(int* err, unsigned long long wait_ns);
int mb_gemm_comm_configure(int* err, unsigned long long wait_ns);
int mb_gemm_rs(const void* X, const void* W, const long long* partial_ptrs, void* out, int* counters, int T, int N, int K, int rank,
               int world, const long long* flag_ptrs, int channel, int epoch, int* error_flag, cudaStream_t s);

#ifdef __cplusplus
}
#endif
