/* C ABI of further sequence mixers of the hybrid decoders (libfa_b200_mixers.so, sm_100a): gated linear recurrences with a matrix
 * state, their gates and short convolution, and grouped-query attention on paged keys and values inside chunks.
 *
 * Conventions: device pointers on the current device; every call is asynchronous on `stream` (a cudaStream_t);
 * nothing is allocated.  `dtype` is the type of activations, weights and cached rows: FAM_F32 or FAM_BF16; states, normalisers,
 * decays and weights of the recurrences are always fp32.  `status` is one int32 in device memory that the caller has set to
 * zero: a kernel that meets a block-table entry or a state slot outside the cache sets bit 1 in it and skips the access; a bounded
 * wait that ran out sets bit 0.  Sequences: slots [n_seq] are the state slots, starts [n_seq] the positions of their first tokens in
 * this call, cu_seqlens [n_seq + 1] their token offsets (null: one token each).  Return value: 0, or a negative code with a text
 * in fam_last_error(). */
#ifndef FA_B200_MIXERS_H
#define FA_B200_MIXERS_H
#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

enum { FAM_F32 = 0, FAM_BF16 = 1 };
enum { FAM_OK = 0, FAM_ERR_INVALID_ARGUMENT = -1, FAM_ERR_UNSUPPORTED = -2, FAM_ERR_CUDA = -4 };

const char* fam_last_error(void);

/* S_t = exp(la_t) S_(t-1) + b_t k_t v_t^T, y_t = S_t^T (q_scale q_t) per head; head h has the queries and keys of group
 * h / (heads / groups).  With `floor`: n_t = exp(la_t) n_(t-1) + b_t k_t, and y_t is divided by max(|n_t . q_t|, floor_t) + norm_eps.  With
 * `skip`: skip_h v_t is added.
 * x [total, stride] holds the groups x dk queries at column off_q, keys at off_k, heads x dv values at off_v; la, b, floor [heads, total];
 * n0 [n_seq, heads, dk] the normaliser before the call; state [n_slots, heads, dk, dv]; norm [n_slots, 2, heads, dk], the normaliser
 * after position p in half p & 1; out [total, heads * dv].  max_len: the longest sequence of the call.  The workspace has
 * fam_recurrence_workspace bytes (0: none is needed). */
typedef struct {
  const void* x;
  int64_t stride, total;
  int32_t off_q, off_k, off_v, heads, groups, dk, dv, n_slots, n_seq, max_len, dtype;
  float q_scale, norm_eps;
  const float *la, *b, *floor, *n0, *skip;
  float *norm, *state;
  const int32_t *slots, *starts, *cu_seqlens;
  void *out, *workspace;
  int64_t workspace_bytes;
  int32_t* status;
} FamRecurrence;
size_t fam_recurrence_workspace(const FamRecurrence* args);
int fam_recurrence(const FamRecurrence* args, void* stream);

/* Exponential gates with a running maximum m (0 before position 0): i = cap tanh((x_i + bias_i) / cap),
 * f = logsigmoid(cap tanh((x_f + bias_f) / cap)), m_t = max(f + m_(t-1), i); la = f + m_(t-1) - m_t, b = exp(i - m_t), floor = exp(-m_t), all
 * [heads, total].  m [n_slots, 2, heads], the maximum after position p in half p & 1; norm, likewise [n_slots, 2, heads, dk], is copied
 * to n0 [n_seq, heads, dk] as it is before the call. */
int fam_max_gates(const void* x, int64_t stride, int off_i, int off_f, int heads, const void* bias_i, const void* bias_f, float cap, float* m,
                  const float* norm, float* n0, int dk, int n_slots, const int32_t* slots, const int32_t* starts, const int32_t* cu_seqlens, int n_seq,
                  int64_t total, float* la, float* b, float* floor, int32_t* status, int dtype, void* stream);

/* dt = softplus(x[:, off + h] + bias_h): la = -exp(a_log_h) dt, b = dt, [heads, total]. */
int fam_step_gates(const void* x, int64_t stride, int off, int heads, const float* bias, const float* a_log, int64_t total, float* la, float* b,
                   int dtype, void* stream);

/* Causal convolution per channel and SiLU: out [total, channels] = silu(bias + sum_k w[taps - 1 - k] x[t - k]), w [taps, channels].  Inputs of
 * earlier calls come from ring [n_slots, taps, channels] (position p in row p % taps; positions before 0 are zero), where the last ones
 * of this call are left. */
int fam_conv_silu(const void* x, int64_t stride, int off, int channels, int taps, const void* w, const void* bias, void* ring, int n_slots,
                  const int32_t* slots, const int32_t* starts, const int32_t* cu_seqlens, const int32_t* tok_seq, const int32_t* positions, int n_seq,
                  int64_t total, void* out, int32_t* status, int dtype, void* stream);

/* Decode steps, one token per sequence, in one kernel each (sizes: fam_recurrence_step_supported).  `args` as fam_recurrence without
 * la, b, floor and n0, which the step computes: with the gates of fam_max_gates, or with the convolution and gates of fam_conv_silu and
 * fam_step_gates, x being the projection with the columns of v, k and q (in this order, adjacent) before the convolution. */
int fam_recurrence_step_supported(int dk, int dv);
int fam_max_gate_step(const FamRecurrence* args, int off_i, int off_f, const void* bias_i, const void* bias_f, float cap, float* m, void* stream);
int fam_ssd_step(const FamRecurrence* args, int off_dt, const float* dt_bias, const float* a_log, const void* conv_w, const void* conv_b, void* ring,
                 int taps, void* stream);

/* Pages: pools [n_blocks, kv_heads, 16, dim] and [n_blocks, kv_heads, 16, vdim] behind block_table [n_seq, max_blocks]; row r of a call is the
 * token at positions[r] of sequence tok_seq[r]. */
typedef struct {
  void *k_pool, *v_pool;
  const int32_t *block_table, *tok_seq, *positions;
  int32_t n_blocks, max_blocks, n_seq, heads, kv_heads, dim, vdim, dtype;
  int64_t rows;
  int32_t* status;
} FamPages;

/* x [rows, stride]: q and k are RMS-normed over all heads' columns at once, v = (1 - lambda) v + lambda v_first where v_first (row stride
 * first_stride) is given; k and v go to their places in the pages and, where given, to k_out and v_out; q to q_out. */
int fam_kv_prep(const FamPages* pages, const void* x, int64_t stride, int off_q, int off_k, int off_v, const void* wq, const void* wk, float eps,
                const void* v_first, int64_t first_stride, float lambda, void* q_out, void* k_out, void* v_out, void* stream);

/* Every row sees the keys from the start of its chunk of `chunk` positions (0: from position 0) to its own; scores
 * scale (q . k) - slopes_h (distance), slopes null: 0.  out (row stride out_stride) = softmax-weighted values times sigmoid(gate) (gate, row
 * stride gate_stride, may be null).  The workspace has fam_kv_attention_workspace bytes (0: none is needed). */
size_t fam_kv_attention_workspace(const FamPages* pages, int chunk);
int fam_kv_attention(const FamPages* pages, const void* q, const float* slopes, const void* gate, int64_t gate_stride, int chunk, float scale, void* out,
                     int64_t out_stride, void* workspace, size_t workspace_bytes, void* stream);

/* Cached rows as contiguous rows: piece i takes the positions from piece_key0[i] on of sequence piece_seq[i], cu_kv [pieces + 1]. */
int fam_kv_gather(const FamPages* pages, const int32_t* piece_seq, const int32_t* piece_key0, const int32_t* cu_kv, int pieces, int64_t total_kv, void* k,
                  void* v, void* stream);

/* Prompt attention on contiguous rows (bfloat16): q [total_q, heads, dim], k [total_kv, kv_heads, dim], v [total_kv, kv_heads, vdim]; a piece's
 * queries are its last keys, causal inside the piece.  Scores, gate and output as fam_kv_attention. */
int fam_kv_prefill_supported(int heads, int kv_heads, int dim, int vdim, float scale, int dtype);
int fam_kv_prefill(const void* q, const void* k, const void* v, const int32_t* cu_q, const int32_t* cu_kv, int pieces, int max_q, int64_t total_q,
                   int64_t total_kv, int heads, int kv_heads, int dim, int vdim, float scale, const float* slopes, const void* gate,
                   int64_t gate_stride, void* out, int64_t out_stride, int32_t* status, void* stream);

#ifdef __cplusplus
}
#endif
#endif
