// C entry points of the sm_100a kernels. Pointers are device pointers; every launcher enqueues on
// `stream` and returns 0 or an error code (cudaError_t value, or a negative code for bad arguments).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

// GEMM epilogue flags
#define GEMM_FLAG_BIAS 1          // + bias[n]
#define GEMM_FLAG_GELU 2          // tanh-GeLU after bias
#define GEMM_FLAG_SAVE_PREACT 4   // also write (acc + bias) to aux_out (needed by the GeLU backward)
#define GEMM_FLAG_DGELU 8         // multiply by gelu'(aux[m,n])
#define GEMM_FLAG_RESIDUAL 16     // + aux[m,n] (aux has the output dtype)
#define GEMM_FLAG_OUT_FP32 32     // D is fp32 (default: same 16-bit type as the inputs)
#define GEMM_FLAG_ACCUMULATE 64   // D += result
#define GEMM_FLAG_FP16 128        // inputs are fp16 (default bf16)
#define GEMM_FLAG_CE_STATS 256    // LM head + cross-entropy, forward: no D; per (row, 128-column block) the epilogue emits
                                  // (max, sum exp(x - max), logit of the row's label if it lies in the block)
#define GEMM_FLAG_CE_GRAD 512     // LM head + cross-entropy, backward: D = (exp(x - lse[row]) - [col == label]) * scale[row]
#define GEMM_FLAG_RELU2 1024      // square of relu
#define OSLO_ACT_RELU2 (-2)       // `gelu_from` of the few-row products: square of relu on all columns
#define GEMM_FLAG_GLU 2048        // columns in pairs (gate, up): silu(gate) * up, half as many output columns; N is even, ldd >= N / 2
#define GEMM_CE_BLOCK 128         // columns per statistics record

#define OSLO_DT_BF16 0
#define OSLO_DT_FP16 1
#define OSLO_DT_FP32 2

#ifdef __cplusplus
extern "C" {
#endif

int oslo_gemm_16bit(const void* A, const void* B, void* D, int M, int N, int K, int lda, int ldb, int ldd,
                    int a_mn_major, int b_mn_major, const void* bias, const void* aux, int ld_aux, void* aux_out,
                    int ld_aux_out, int flags, float alpha, int* err_word, int num_sms, cudaStream_t stream);

// LM-head product with the cross-entropy pieces in its epilogue (x = A B^T + bias, never written as logits):
//   mode 0 (GEMM_FLAG_CE_STATS): stats [ceil(N / 128), M, 3] fp32 records (max, sum exp, label logit or 0)
//   mode 1 (GEMM_FLAG_CE_GRAD):  D [M, N] (input dtype) = (softmax - onehot) * scale, from lse / scale fp32 [M]
// labels int64 [M] are global vocabulary ids; this rank's columns are ids vocab_start .. vocab_start + N - 1
int oslo_gemm_ce_16bit(const void* A, const void* B, int M, int N, int K, int lda, int ldb, int b_mn_major,
                       const void* bias, const long long* labels, long long vocab_start, int mode, float* stats,
                       const float* lse, const float* scale, void* D, int ldd, int fp16, int* err_word, int num_sms,
                       cudaStream_t stream);
// (max, sum exp, label logit) per row from the per-block records of mode 0
int oslo_ce_reduce_stats(const float* stats, float* rowmax, float* sumexp, float* target, int rows, int blocks,
                         cudaStream_t stream);

// few-row GEMM for decode steps (M <= 128): k range cut into `split_k` slices, slice s writes its fp32 partial sums
// to plane s of D [split_k, M, N]; oslo_gemm_split_k_for suggests the slice count (1 = use oslo_gemm_16bit)
int oslo_gemm_split_k_for(int M, int N, int K, int num_sms);
int oslo_gemm_splitk_16bit(const void* A, const void* B, float* D, int M, int N, int K, int lda, int ldb, int ldd,
                           int a_mn_major, int b_mn_major, int fp16, int split_k, int* err_word, int num_sms,
                           cudaStream_t stream);
// out = T(act(sum over planes of ws + bias)) for the [split_k, rows, cols] fp32 result of the split-K GEMM;
// tanh-GeLU on columns >= gelu_from (-1 = none)
int oslo_splitk_finalize(const float* ws, const void* bias, void* out, long long rows, int cols, int split_k,
                         int gelu_from, int dtype, cudaStream_t stream);

// LayerNorm over the last dim of [rows, cols]; mean/rstd are fp32 [rows]
int oslo_layernorm_fwd(const void* x, const void* w, const void* b, void* y, float* mean, float* rstd, int rows,
                       int cols, float eps, int dtype, cudaStream_t stream);
// dw/db partial sums: [parts, cols] fp32 workspaces, reduced by a second kernel into dw/db (input dtype)
int oslo_layernorm_bwd(const void* dy, const void* x, const void* w, const float* mean, const float* rstd, void* dx,
                       float* dw_part, float* db_part, void* dw, void* db, int rows, int cols, int parts, int dtype,
                       cudaStream_t stream);

int oslo_bias_gelu_fwd(const void* x, const void* bias, void* y, long long rows, int cols, int dtype,
                       cudaStream_t stream);
int oslo_bias_gelu_bwd(const void* dy, const void* x, const void* bias, void* dx, long long rows, int cols, int dtype,
                       cudaStream_t stream);
// y = dropout(x + bias) + residual; the keep-mask is a counter hash of (seed, element index), so backward
// regenerates it instead of storing it. mode 0 = forward, 1 = backward (x is dy; bias/residual ignored)
int oslo_bias_dropout_residual(const void* x, const void* bias, const void* residual, void* y, long long rows,
                               int cols, float p, unsigned long long seed, int mode, int dtype, cudaStream_t stream);
// column sums of [rows, cols] into fp32 [cols] (bias gradients); part is a [parts, cols] workspace
int oslo_colsum(const void* x, float* part, float* out, int rows, int cols, int parts, int dtype,
                cudaStream_t stream);

// GPT-J rotary on [B, S, heads, D] (contiguous), pairs (2i, 2i+1) of the first rotary_dim dims; positions
// int64 [B, S]; inverse = 1 applies the transpose rotation (backward)
int oslo_rotary(const void* x, void* y, const long long* positions, int B, int S, int H, int D, int rotary_dim,
                float base, int inverse, int dtype, cudaStream_t stream);

// same rotation applied in place; touches only the first rotary_dim dims of each head (rotary_dim % 8 == 0, D % 8 == 0)
int oslo_rotary_inplace(void* x, const long long* positions, int B, int S, int H, int D, int rotary_dim, float base,
                        int inverse, int dtype, cudaStream_t stream);

// softmax on materialised scores
int oslo_causal_softmax_fwd(const void* x, void* y, int batches, int sq, int sk, float scale, int dtype,
                            cudaStream_t stream);
int oslo_masked_softmax_fwd(const void* x, const uint8_t* mask, void* y, int b, int h, int sq, int sk,
                            int mask_b, float scale, int dtype, cudaStream_t stream);
int oslo_softmax_bwd(const void* y, const void* dy, void* dx, long long rows, int cols, float scale, int dtype,
                     cudaStream_t stream);

// cross-entropy pieces over logits [rows, cols] (16-bit or fp32), labels int64 shifted by vocab_start
int oslo_ce_stats(const void* logits, const long long* labels, float* rowmax, float* sumexp, float* target,
                  int rows, int cols, int ld, long long vocab_start, int dtype, cudaStream_t stream);
int oslo_ce_grad(void* logits, const long long* labels, const float* lse, const float* scale, int rows, int cols,
                 int ld, long long vocab_start, int dtype, cudaStream_t stream);

// AdamW on flat buffers: fp32 master p, 16-bit or fp32 grads, optional 16-bit copy of the new params
int oslo_adam(float* p, const void* g, float* m, float* v, void* p_lp, long long n, float lr, float beta1,
              float beta2, float eps, float wd, float bc1, float bc2, float grad_scale, const float* inv_scale_dev,
              int g_dtype, int lp_dtype, cudaStream_t stream);
// sum of squares of a flat buffer into out[0] (atomic add; zero it first)
int oslo_sumsq(const void* x, float* out, long long n, int dtype, cudaStream_t stream);

// n-gram repeat blocking: lprobs[row, tok] = -inf for tokens that would complete a seen n-gram
int oslo_ngram_ban(const long long* tokens, float* lprobs, int rows, int len, int vocab, int n, int* err_word,
                   cudaStream_t stream);

// flash attention. q/k/v/o: element strides for (batch, head, seq); last dim contiguous
int oslo_flash_fwd(const void* q, const void* k, const void* v, void* o, float* lse, const uint8_t* kpm, int B,
                   int H, int Sq, int Sk, int D, long long q_sb, long long q_sh, long long q_ss, long long k_sb,
                   long long k_sh, long long k_ss, long long v_sb, long long v_sh, long long v_ss, long long o_sb,
                   long long o_sh, long long o_ss, float scale, int causal, int window, int dtype,
                   cudaStream_t stream);
// same contract as oslo_flash_fwd, on the tcgen05 tensor cores with TMEM accumulators (attention_sm100.cu)
int oslo_flash_fwd_sm100(const void* q, const void* k, const void* v, void* o, float* lse, const uint8_t* kpm, int B,
                         int H, int Sq, int Sk, int D, long long q_sb, long long q_sh, long long q_ss, long long k_sb,
                         long long k_sh, long long k_ss, long long v_sb, long long v_sh, long long v_ss, long long o_sb,
                         long long o_sh, long long o_ss, float scale, int causal, int window, int dtype, int* err_word,
                         cudaStream_t stream);
// causal, with exp(sink[h]) in the denominator and a sigmoid output gate per (position, head); stores the first d_out columns
int oslo_flash_sink_fwd_sm100(const void* q, const void* k, const void* v, void* o, const uint8_t* kpm, const void* sink,
                              const void* gate, long long ldg, int B, int H, int G, int Sq, int Sk, int dim, int vdim,
                              long long q_sb, long long q_sh, long long q_ss, long long k_sb, long long k_sh, long long k_ss,
                              long long v_sb, long long v_sh, long long v_ss, long long o_sb, long long o_sh, long long o_ss,
                              float scale, float softcap, int window, int keep_first, const int* lead, int gate_wide,
                              const void* q2, long long q2_sb, long long q2_sh, long long q2_ss, const void* k2, long long k2_sb,
                              long long k2_ss, int rot, int dtype, int* err_word, cudaStream_t stream);
// the same with one key head of any width for all query heads, k [B, Sk, dim], and value heads per group
int oslo_flash_wide_fwd_sm100(const void* q, const void* k, const void* v, void* o, const uint8_t* kpm, const void* sink,
                              const void* gate, long long ldg, int gate_wide, int B, int H, int G, int Sq, int Sk, int dim, int vdim,
                              long long q_sb, long long q_sh, long long q_ss, long long k_sb, long long k_ss, long long v_sb,
                              long long v_sh, long long v_ss, long long o_sb, long long o_sh, long long o_ss, float scale, int window,
                              int keep_first, const int* lead, int dtype, int* err_word, cudaStream_t stream);
int oslo_flash_bwd(const void* q, const void* k, const void* v, const void* o, const void* dout, const float* lse,
                   float* delta, float* dq_acc, void* dq, void* dk, void* dv, const uint8_t* kpm, int B, int H,
                   int Sq, int Sk, int D, long long q_sb, long long q_sh, long long q_ss, long long k_sb,
                   long long k_sh, long long k_ss, long long v_sb, long long v_sh, long long v_ss, long long o_sb,
                   long long o_sh, long long o_ss, long long do_sb, long long do_sh, long long do_ss, float scale,
                   int causal, int window, int dtype, cudaStream_t stream);
// same contract on the tcgen05 tensor cores (attention_bwd_sm100.cu); dq / dk / dv use the strides of q / k / v
int oslo_flash_bwd_sm100(const void* q, const void* k, const void* v, const void* o, const void* dout, const float* lse,
                         float* delta, void* dq, void* dk, void* dv, const uint8_t* kpm, int B, int H, int Sq, int Sk,
                         int D, long long q_sb, long long q_sh, long long q_ss, long long k_sb, long long k_sh,
                         long long k_ss, long long v_sb, long long v_sh, long long v_ss, long long o_sb, long long o_sh,
                         long long o_ss, long long do_sb, long long do_sh, long long do_ss, float scale, int causal,
                         int window, int dtype, int* err_word, cudaStream_t stream);
// single-query attention over a static cache [B, H, T, D]; lengths int32 [B]
int oslo_decode_attn(const void* q, const void* kc, const void* vc, void* o, const int* lengths, float* ws, int B,
                     int H, int T, int D, int splits, float scale, int window, int dtype, int* err_word,
                     cudaStream_t stream);

// GEMM fused with a tensor-parallel collective (fused_comm_gemm.cu); mode 1 = all-reduce (result left in the
// symmetric staging matrix), 2 = reduce-scatter into out, 3 = all-gather of A then GEMM into out
// aux / ld_aux: with GEMM_FLAG_RESIDUAL in the reduce modes, another per-rank partial sum [M, N] added before the reduction
int oslo_gemm_comm_16bit(const void* A, const void* B, int M, int N, int K, int lda, int ldb, int a_mn_major,
                         int b_mn_major, const void* bias, const void* aux, int ld_aux, void* aux_out, int ld_aux_out,
                         int flags, float alpha,
                         void* const* peer_bufs_dev, void* own_buf, void* mc_base, long long data_off,
                         long long flag_off, long long flag_bytes, int rank, int world, unsigned epoch,
                         unsigned done_base, int mode, int use_multimem, void* out, int ld_out, int wide_tiles,
                         unsigned long long* trace, int* err_word, int num_sms, cudaStream_t stream);

// symmetric-memory collectives (comm.cu)
int oslo_allreduce_symm(void* const* peer_ptrs_dev, void* mc_ptr, uint32_t* const* signal_ptrs_dev, void* out,
                        long long n, int rank, int world, int dtype, int use_multimem, int* err_word,
                        cudaStream_t stream);

// data-parallel reduce-scatter / all-gather of one bucket [lo, hi) (16-bit elements) of a symmetric flat buffer whose
// rank r owns [r * shard, (r + 1) * shard); in place (comm.cu)
int oslo_dp_reduce_scatter(void* const* peer_ptrs_dev, void* mc_ptr, uint32_t* const* signal_ptrs_dev, long long lo,
                           long long hi, long long shard, int rank, int world, int dtype, int use_multimem,
                           int* err_word, cudaStream_t stream);
int oslo_dp_all_gather(void* const* peer_ptrs_dev, void* mc_ptr, uint32_t* const* signal_ptrs_dev, long long lo,
                       long long hi, long long shard, int rank, int world, int use_multimem, int* err_word,
                       cudaStream_t stream);

// vocabulary-parallel cross-entropy: combine every rank's per-row (max, sum exp, label logit) over the group in one
// kernel through a symmetric staging buffer of 2 x 3 x cap floats (comm.cu)
int oslo_ce_combine(const float* mx, const float* se, const float* tg, float* out_mx, float* out_se, float* out_tg,
                    void* const* peer_ptrs_dev, uint32_t* const* signal_ptrs_dev, uint32_t* counters, int n, int cap,
                    int rank, int world, int* err_word, cudaStream_t stream);

// decode-step kernels (decode_sm100.cu). gemv_rows: out[m, n] = act([x1 | x2][m, :] . W[n, :] + bias[n]) for M <= 4
// rows, W [N, K1 + K2] K-major, tanh-GeLU on columns >= gelu_from (-1 = none); x2 may be null.
// `res` [M, N] (row stride ldr) is added after the activation; bias and res may be null.
// P of them at once: x [P, M, K] and W [P, N, K] (strides sx, sw between parts) -> out [P, M, N]
int oslo_gemv_stacked(const void* x, int ldx, long long sx, const void* W, int ldw, long long sw, void* out, int P, int M, int N, int K,
                      int dtype, int num_sms, cudaStream_t stream);
int oslo_gemv_rows(const void* x1, int ld1, int K1, const void* x2, int ld2, int K2, const void* W, int ldw,
                   const void* bias, const void* res, int ldr, void* out, int ldo, int M, int N, int gelu_from,
                   int dtype, int num_sms, cudaStream_t stream);
// rotary on the new token's q and k, q -> q_out [B, H, D], k / v -> cache [B, H, Tmax, D] at write_index[0];
// the rotary position of row b is lengths[b]
int oslo_rotary_append(const void* q, const void* k, const void* v, long long ldq, long long ldk, long long ldv,
                       void* q_out, void* kc, void* vc, const int* lengths, const long long* write_index, int B, int H,
                       int D, int Tmax, int rotary_dim, float base, int dtype, int* err_word, cudaStream_t stream);

// vocab-parallel embedding lookup + its collective in one kernel (comm.cu): the owner of a token's row stores it into
// every rank's staging half of the symmetric buffer, one cross-rank barrier, copy-out
int oslo_vocab_embed(const long long* ids, const void* weight, void* out, void* const* peer_ptrs_dev, void* mc_ptr,
                     uint32_t* const* signal_ptrs_dev, uint32_t* counters, long long tokens, int H, long long lo,
                     long long hi, long long half_bytes, int rank, int world, int dtype, int use_multimem, int* err_word,
                     int num_sms, cudaStream_t stream);

// bounded wait on a local flag with a caller-chosen limit (<= 1 s); for tests of the give-up path (comm.cu)
int oslo_wait_probe(const uint32_t* flag, uint32_t target, unsigned long long limit_ns, int* err_word,
                    unsigned long long* waited_ns, cudaStream_t stream);

// one-kernel all-reduce for small tensors (comm.cu): in -> staging half in symmetric memory -> sum over ranks -> out
int oslo_allreduce_oneshot(const void* in, void* out, void* const* peer_ptrs_dev, void* mc_ptr,
                           uint32_t* const* signal_ptrs_dev, uint32_t* counters, long long n, long long stage_off,
                           long long half_bytes, int rank, int world, int dtype, int use_multimem, int* err_word,
                           cudaStream_t stream);

// RMS norms and the residual join (rms_norm.cu). x is fp32 when x_fp32, else the storage type; rows have strides;
// one: the weight is one number
int oslo_rms_norm(const void* x, long long ldx, int x_fp32, const void* w, int one, void* out, long long ldo, long long rows, int cols,
                  float eps, float offset, int dtype, cudaStream_t stream);
// x_out = x + rms(y * sigmoid(gate + gate_bias)) * (1 + w_post); h_out = rms(x_out) * (1 + w_next) unless w_next is null.
// slot_weights null: y has one row per token, else y = sum_j slot_weights[t, j] * y[slots[t, j]] (slots null: t * top + j)
int oslo_residual_join(const float* x, const void* y, long long ldy, const int* slots, const float* slot_weights, int top,
                       const void* gate, long long ldg, const void* gate_bias, const void* w_post, const void* w_next,
                       float* x_out, void* h_out, long long rows, int cols, float eps, int dtype, cudaStream_t stream);
int oslo_silu_mul(const void* gate, long long ldg, const void* up, long long ldu, void* out, long long rows, int cols, int dtype,
                  cudaStream_t stream);
// g sigmoid(alpha g) (u + 1), g = min(gate, limit), u = clamp(up, -limit, limit)
int oslo_clamped_glu(const void* gate, long long ldg, const void* up, long long ldu, void* out, long long rows, int cols,
                     float limit, float alpha, int dtype, cudaStream_t stream);
// x_out = x + mult * sum_i factor[i] * b_i, i < n <= 3, with b_i = y[i], rms(y[i]) * w[i] (normed) or y[i] * w[i]; top[i] > 0: y[i] of a
// row is the sum of the rows slots[i][row, j] (null: row * top + j), j < top. h1 = rms(x_out) * w1, h2 = rms(x_out) * w2 (w2 or both null:
// not written; one1, one2: the weight is one number); copy (w1 null): h1 = x_out. conv_w [cols, taps] (rows are single tokens):
// conv_out = h1 + the causal convolution of prev fp32 [rows, taps - 1, cols] and h1, prev moves on (null: zeros); keep 0: h1 counts as 0
struct OsloBranchJoin {
  const float* x; int n;
  const void* y[3]; long long ldy[3]; const void* w[3]; int normed[3]; const int* slots[3]; int top[3]; float factor[3];
  float mult, eps;
  const void *w1, *w2; int one1, one2, copy;
  float* x_out; void *h1, *h2;
  const void* conv_w; float* prev; int taps; const uint8_t* keep; long long ld_keep; void* conv_out;
};
int oslo_branch_join(const struct OsloBranchJoin* a, long long rows, int cols, int dtype, cudaStream_t stream);
// out [rows, cols] = gelu_tanh(z) * table[ids[row * id_step], first + column]
int oslo_token_gate(const void* z, long long ldz, const long long* ids, long long id_step, const void* table, long long ldt,
                    long long vocab, int first, void* out, long long rows, int cols, int dtype, int* err_word, cudaStream_t stream);
// out = o / rms(runs of `group` columns) * w * act(gate); act 0: sigmoid, 1: silu; o fp32 [rows, cols]
// z, m [rows, cols / group] (or null): the runs are first divided by max(|z|, exp(-m)) + 1e-6
int oslo_gated_rms_norm(const float* o, const void* w, const void* gate, long long ldg, void* out, const float* z, const float* m,
                        long long rows, int cols, int group, float eps, int act, int dtype, cudaStream_t stream);

// residual streams (hyper_connections.cu): x [rows, n, cols] fp32 with row and stream strides, x_out contiguous, h [rows, cols].
// y null: the streams stay. weights null: y has one row per token, else y = sum_j weights[t, j] * row, which is y's row slots[t, j]
// (null: t * top + j) or, where choice[t, j] >= experts, own's row t. shared null or added times sigmoid(gate). w_in null: ones
int oslo_hyper_join(const float* x, long long x_row, long long x_stream, const void* y, long long ldy, const int* slots,
                    const float* weights, int top, const int* choice, int experts, const void* own, long long ld_own,
                    const void* shared, long long ld_shared, const void* gate, long long ld_gate, const void* w_out, const void* mix,
                    const void* w_in, const void* w_norm, float* x_out, void* h, long long rows, int n, int cols, float eps,
                    float scale, int dtype, cudaStream_t stream);

// linear recurrences (linear_recurrence.cu): q, f [B * S, H * dim], v [B * S, H * vdim] with row strides; keep [B, S]
// (0 = padding) or null; state [B, H, dim, vdim] fp32, read and updated, or null; out fp32 [B, S, H, vdim].
// nchunks > 1 (oslo_recurrence_chunks) needs ws [B, nchunks, H, dim, vdim] and decay [B, nchunks, H, dim] fp32.
// rule 0: f are forget-gate logits with f_bias and lower bounds [H * dim]; 1: f are keys, head_decay [H] fp32; 2: f are keys,
// f_bias = w0 and lower = u [H * dim], z the decay logits fp32 [B * S, H * dim]
int oslo_recurrence_chunks(int rule, int B, int S, int H, int dim, int vdim, int num_sms);
int oslo_recurrence(int rule, const void* q, long long ldq, const void* f, long long ldf, const void* v, long long ldv,
                    const void* f_bias, const void* lower, const float* z, long long ldz, const float* head_decay,
                    const uint8_t* keep, long long ld_keep, float* state, float* out, float* ws, float* decay, int nchunks, int B,
                    int S, int H, int dim, int vdim, int dtype, cudaStream_t stream);
// one token per row, the outputs RMS-normed per head with norm_w [vdim]
int oslo_recurrence_step(const void* q, long long ldq, const void* f, long long ldf, const void* v, long long ldv,
                         const void* f_bias, const void* lower, const void* norm_w, const uint8_t* keep, long long ld_keep,
                         float* state, void* out, float eps, int B, int H, int dim, int vdim, int num_sms, int dtype, cudaStream_t stream);

// rule 1, one token per row: out fp32 [B, H * vdim], not normed
int oslo_decayed_step(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                      const float* head_decay, const uint8_t* keep, long long ld_keep, float* state, float* out, int B, int H,
                      int dim, int vdim, int num_sms, int dtype, cudaStream_t stream);
// rule 2, one token per row: decay logits W_w2 tanh(t) (t [B, rank], w2 [H * dim, rank]), heads RMS-normed, times norm_w
// [H * vdim] and silu(gate)
int oslo_bonus_step(const void* r, long long ldr, const void* k, long long ldk, const void* v, long long ldv, const void* t,
                    long long ldt, const void* w2, int rank, const void* w0, const void* u, const void* norm_w, const void* gate,
                    long long ldg, const uint8_t* keep, long long ld_keep, float* state, void* out, float eps, int B, int H, int dim,
                    int vdim, int num_sms, int dtype, cudaStream_t stream);

// rule 3 (matrix memory): state [B, H, dim, lds], lds = vdim + 1 rounded up to a multiple of 4, column vdim the normaliser; read,
// write, start [B, H, S] of oslo_memory_gates; norm [B, S, H]; ws [B, nchunks, H, dim, lds]
int oslo_memory_recurrence(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const float* read,
                           const float* write, const float* start, float q_scale, const uint8_t* keep, long long ld_keep, float* state,
                           float* out, float* norm, float* ws, float* decay, int nchunks, int B, int S, int H, int dim, int vdim,
                           int dtype, cudaStream_t stream);
// matrix_memory.cu: z fp32 [B * S, 2 H], bias [2 H], top [B, H] (read and updated) or null, m_out [B, S, H]
int oslo_memory_gates(const float* z, long long ldz, const void* bias, float cap, const uint8_t* keep, long long ld_keep, float* top,
                      float* read, float* write, float* start, float* m_out, int B, int S, int H, int dtype, cudaStream_t stream);
// one token per row: gates from x [B, width], memory, normaliser, head norms with norm_w [H * vdim], sigmoid(gate)
int oslo_memory_step(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const void* x, long long ldx,
                     int width, const void* w, const void* bias, float cap, const void* gate, long long ldg, const void* norm_w,
                     const uint8_t* keep, long long ld_keep, float* state, float* top, void* out, float q_scale, float eps, int B, int H,
                     int dim, int vdim, int num_sms, int dtype, cudaStream_t stream);

// latent attention (latent_attention.cu). sink_gate: flash output [B, S, H, *] + lse [B, H, S] -> out [B * S, H * vdim]
int oslo_sink_gate(const void* o, long long o_sb, long long o_ss, long long o_sh, const float* lse, const void* sink,
                   const void* gate, long long ldg, void* out, int B, int S, int H, int vdim, int dtype, cudaStream_t stream);
// causal attention with sink and output gate (or null) in 32-bit, any head sizes; strides of (batch, position, head); KG key and G
// value heads; softcap > 0: scores become softcap * tanh(score / softcap)
int oslo_sink_attention(const void* q, long long q_sb, long long q_ss, long long q_sh, const void* k, long long k_sb,
                        long long k_ss, long long k_sh, const void* v, long long v_sb, long long v_ss, long long v_sh,
                        const uint8_t* keep, long long ld_keep, const void* sink, const void* gate, long long ldg, void* out,
                        int B, int H, int G, int KG, int Sq, int Sk, int dim, int vdim, float scale, float softcap, int window,
                        int keep_first, const int* lead, int gate_wide, int dtype, cudaStream_t stream);
// rows b * S + t: RMS norm of the query latent -> cq_out; of the key-value latent (null: none) -> cache [B, Tmax, kv_rank + rot] at
// lengths[b] + t, followed by the rot columns after it, rotated (halves) by pos[b, t] * freq; c_out (null: none) [B * S, kv_rank]
// gets the normed latents once more
int oslo_latent_prep(const void* cq, long long ldq, const void* wq, int q_rank, void* cq_out, const void* ckv, long long ldkv,
                     const void* wkv, int kv_rank, void* cache, const int* lengths, int Tmax, float eps, int B, int S, int rot,
                     const long long* pos, long long pos_sb, long long pos_ss, const float* freq, void* c_out, int dtype,
                     int* err_word, cudaStream_t stream);
// in place: the last rot dims of every head of q [B * S, H * (dim + rot)] (contiguous) turn by pos[b, t] * freq, halves paired
int oslo_rotate_halves(void* q, const long long* pos, long long pos_sb, long long pos_ss, const float* freq, int B, int S, int H,
                       int dim, int rot, int dtype, cudaStream_t stream);
// one query per row, q [B, H * (dim + rot)], over a latent cache [B, Tmax, R + rot]; the query's last rot dims are rotated by pos[b] *
// freq; sink null: none; gate_wide: a gate per output element; fp32 workspaces qa [B, H, R + rot], ws [B, H, splits, R rounded up
// to a multiple of 4] and stat [B, H, splits, 2]
int oslo_latent_decode(const void* q, long long ldq, const void* w_uk, long long ldk, const void* w_uv, long long ldv,
                       const void* cache, const int* lengths, const uint8_t* keep, long long ld_keep, int n_keep,
                       const void* sink, const void* gate, long long ldg, float* qa, float* ws, float* stat, void* out,
                       int B, int H, int dim, int vdim, int R, int rot, const long long* pos, long long pos_sb, const float* freq,
                       int gate_wide, int Tmax, int splits, float scale, int num_sms, int dtype, int* err_word,
                       cudaStream_t stream);
int oslo_latent_splits(int B, int H, int T, int num_sms);

// grouped-query attention (grouped_attention.cu). qkv_prep: RMS norm of every query / key head (weights wq, wk [dim] or null), rotation of
// the first 2 * n_freq dims by pos[b, t] * freq, q -> q_out [B, S, H, dim], k / v -> caches [B, G, Tmax, *] at lengths[b] + t
int oslo_qkv_prep(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const void* wq,
                  const void* wk, float eps, const long long* pos, long long pos_sb, long long pos_ss, const float* freq, int n_freq,
                  void* q_out, void* kc, void* vc, const int* lengths, int B, int S, int H, int G, int dim, int vdim, int Tmax,
                  int dtype, int* err_word, cudaStream_t stream);
// the same with interleaved pairs or (halves) dims i and i + n_freq, sines and cosines times amplitude; caches by strides of (batch,
// head, position); talk [H, H] or null: the queries of mixed scores for keys of all heads in a row, q_out [B, S, H, G * dim]
int oslo_head_prep(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const void* wq,
                   const void* wk, float eps, const long long* pos, long long pos_sb, long long pos_ss, const float* freq, int n_freq,
                   int halves, float amplitude, const void* talk, void* q_out, void* kc, long long k_sb, long long k_sg, long long k_st,
                   void* vc, long long v_sb, long long v_sg, long long v_st, const int* lengths, int B, int S, int H, int G, int dim,
                   int vdim, int Tmax, int num_sms, int dtype, int* err_word, cudaStream_t stream);
// one query per row: q [B, H, dim], caches [B, G, Tmax, *], of which lengths[b] positions count; keep [B, n_keep] (0 = padded) or
// null; sink null: none; gate null, [B, H] or (gate_wide) [B, H * vdim / VG]; VG > 1 (G = 1): a cached value row holds VG value heads
// side by side and a query head's result is that of its own; window > 0: the last `window` positions and the first keep_first after lead[b] (null: 0)
// are read; fp32 workspaces ws [B, H, splits, vdim rounded up to a multiple of 4] and stat [B, H, splits, 2]; out [B, H * vdim]
int oslo_grouped_splits(int B, int H, int G, int VG, int T, int dim, int vdim, int dtype, int num_sms);
int oslo_wide_decode_fits(int H, int VG, int dim, int vdim, int dtype);
int oslo_grouped_decode(const void* q, const void* kc, const void* vc, const int* lengths, const uint8_t* keep, long long ld_keep,
                        int n_keep, const void* sink, const void* gate, long long ldg, int gate_wide, int window, int keep_first,
                        const int* lead, float* ws, float* stat, void* out, int B, int H, int G, int VG, int dim, int vdim, int Tmax,
                        int splits, float scale, float softcap, int dtype, int* err_word, cudaStream_t stream);

// token shift, causal convolution and selective scan (selective_scan.cu)
// out[i] = h + (h' - h) * mu[i], i < P; prev fp32 [B, width] (the row before the first; read and updated) or null
int oslo_token_shift(const void* h, long long ldh, const void* mu, const uint8_t* keep, long long ld_keep, float* prev, void* out,
                     int B, int S, int width, int P, int dtype, cudaStream_t stream);
// out [B * S, C] = y = conv(x) + bias (or null), silu(y) or y + x; prev fp32 [B, taps - 1, C] (read and updated) or null
int oslo_causal_conv(const void* x, long long ldx, const void* w, const void* bias, const uint8_t* keep, long long ld_keep, float* prev,
                     void* out, int B, int S, int C, int taps, int silu, int residual, int dtype, cudaStream_t stream);
// dt fp32 logits [B * S, C]; state fp32 [B, C, N] (read and updated) or null; out [B * S, C]. nchunks > 1 (oslo_scan_chunks) needs
// ws [B, nchunks, C, N] and steps [B, nchunks, C] fp32
int oslo_scan_chunks(int B, int S, int C, int N, int num_sms);
int oslo_selective_scan(const void* x, long long ldx, const float* dt, long long lddt, const void* dt_bias, const void* a_log,
                        const void* b, long long ldb, const void* c, long long ldc, const void* d, const void* z, long long ldz,
                        const uint8_t* keep, long long ld_keep, float* state, void* out, float* ws, float* steps, int nchunks, int B,
                        int S, int C, int N, int num_sms, int dtype, cudaStream_t stream);
// one token per row; the step logits are w_dt [C, rank] . dt [B, rank]
int oslo_scan_step(const void* x, long long ldx, const void* dt, long long lddt, const void* w_dt, int rank, const void* dt_bias,
                   const void* a_log, const void* b, long long ldb, const void* c, long long ldc, const void* d, const void* z,
                   long long ldz, const uint8_t* keep, long long ld_keep, float* state, void* out, int B, int C, int N, int dtype,
                   cudaStream_t stream);

// mixture of experts (moe.cu, grouped GEMM in gemm_sm100.cu)
// route: idx, wgt [rows, top]; scored 1: scores are the softmax over all E outputs, bias only enters the choice, weights are the chosen
// scores over their sum; 2: the weights are the sigmoids of the largest logits; bias null: none. Choices >= the experts of plan / few
// get no slot (-1) and no product. unit: 0 none, 1 relu^2, 2 silu(gate) * up of column pairs (out has N / 2 columns), 3 the clamped
// form of that (limit, alpha). scale [pairs] (or null) multiplies what an expert reads
int oslo_moe_route(const void* h, long long ldh, const void* w, const void* bias, const float* logits, long long ldl, int* idx,
                   float* wgt, long long rows, int E, int K, int top, int scored, int dtype, cudaStream_t stream);
int oslo_moe_plan(const void* h, long long ldh, const int* idx, int* cursor, int* tile_group, int* n_tiles, int* slots, void* rows_out,
                  const float* scale, long long pairs, int E, int K, int top, int max_tiles, int dtype, cudaStream_t stream);
int oslo_moe_grouped(const void* a, const void* w, void* out, const int* tile_group, const int* n_tiles, int max_tiles, int N,
                     int K, int unit, float limit, float alpha, int dtype, cudaStream_t stream);
int oslo_moe_few(const void* x, long long ldx, const int* idx, const void* w, void* out, int pairs, int per_row, int N, int K,
                 int unit, float limit, float alpha, const float* scale, int E, int dtype, cudaStream_t stream);
int oslo_gemm_grouped(const void* A, const void* B, void* D, int M, int N, int K, int groups, const int* group_of_tile,
                      const int* group_tiles, int flags, int glu_clamped, float glu_limit, float glu_alpha, int* err_word, int num_sms,
                      cudaStream_t stream);

#ifdef __cplusplus
}
#endif
