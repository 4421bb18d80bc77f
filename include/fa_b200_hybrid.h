/* C ABI of the hybrid decoder's operators (libfa_b200_hybrid.so, sm_100a): decayed linear attention and attention over
 * cached latent rows.  (The row-wise operators between the matrix products: fa_b200_rows.h.)
 *
 * Conventions: device pointers on the current device; every call is asynchronous on `stream` (a cudaStream_t);
 * nothing is allocated.  `dtype` is the type of activations, weights and cached latent rows: FAH_F32 or FAH_BF16; the
 * residual stream and the linear-attention state are always fp32.  `status` is one int32 in device memory that the
 * caller has set to zero: a kernel that meets a block-table entry or a state slot outside the cache sets bit 1 in it
 * and skips the access; a bounded wait that ran out sets bit 0.  Return value: 0, or a negative code with a text in
 * fah_last_error(). */
#ifndef FA_B200_HYBRID_H
#define FA_B200_HYBRID_H
#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

enum { FAH_F32 = 0, FAH_BF16 = 1 };
enum { FAH_OK = 0, FAH_ERR_INVALID_ARGUMENT = -1, FAH_ERR_UNSUPPORTED = -2, FAH_ERR_CUDA = -4 };

const char* fah_last_error(void);

/* Decayed linear attention with SiLU on q, k, v: per head S = decay * S + k v^T, o = S^T q.
 * qkv [tokens, stride] with the heads x dk queries at column off_q, keys at off_k, heads x dv values at off_v;
 * state [n_slots, heads, dk, dv] fp32; out [tokens, heads * dv].  cu_seqlens null: one token per sequence.
 * Prompts (cu_seqlens given) take a workspace of fah_lightning_workspace bytes; max_len is the longest sequence of the call. */
size_t fah_lightning_workspace(int n_seq, int heads, int dk, int dv, int max_len, int dtype);
int fah_lightning(const void* qkv, int64_t stride, int off_q, int off_k, int off_v, int heads, int dk, int dv, const float* decay,
                  float* state, int n_slots, const int32_t* slots, const int32_t* starts, const int32_t* cu_seqlens, int n_seq,
                  int max_len, int64_t tokens, void* out, void* workspace, size_t workspace_bytes, int32_t* status, int dtype,
                  void* stream);

/* down [rows, down_stride]: the query latent at off_q, the key/value latent at off_kv and the shared key part at off_r.
 * cq [rows, q_rank] and the latent c are RMS-normed, the shared part is rotated with cos / sin [rows, rot_dim / 2]; (c, rotated
 * part) go to the row's place in pool [n_blocks, 16, pool_stride] and, where given, to c_out [rows, kv_rank] and
 * r_out [rows, rot_dim]. */
int fah_latent_prep(const void* down, int64_t down_stride, int off_q, int q_rank, int off_kv, int kv_rank, int off_r, int rot_dim,
                    const void* wq, const void* wkv, float eps, const float* cos_t, const float* sin_t, void* cq, void* c_out,
                    void* r_out, void* pool, int pool_stride, int n_blocks, const int32_t* block_table, int max_blocks, int n_seq,
                    const int32_t* tok_seq, const int32_t* positions, int64_t rows, int32_t* status, int dtype, void* stream);

/* Rotates columns [off, off + rot_dim) of every head of q [rows, heads * head_stride] in place (column i pairs with
 * i + rot_dim / 2). */
int fah_rotate_heads(void* q, const float* cos_t, const float* sin_t, int64_t rows, int heads, int head_stride, int off,
                     int rot_dim, int dtype, void* stream);

/* Attention over cached latent rows: every row of (q_abs [rows, heads, kv_rank] | rotated columns
 * [q_off, q_off + rot_dim) of q [rows, heads, q_stride]) sees the keys 0 .. positions[row] of its sequence; values are the
 * latents; the result times sigmoid(gate[row, head]) (gate may be null) goes to out [rows, heads, kv_rank].  The workspace has
 * fah_latent_attention_workspace bytes (0: none is needed). */
size_t fah_latent_attention_workspace(int heads, int kv_rank, int rot_dim, int64_t rows, int dtype);
int fah_latent_attention(const void* q_abs, const void* q, int q_stride, int q_off, const float* cos_t, const float* sin_t,
                         const void* pool, int pool_stride, int n_blocks, const int32_t* block_table, int max_blocks, int n_seq,
                         const int32_t* tok_seq, const int32_t* positions, const void* gate, int64_t gate_stride, int heads,
                         int kv_rank, int rot_dim, float scale, void* out, int64_t rows, void* workspace, size_t workspace_bytes,
                         int32_t* status, int dtype, void* stream);

/* Prompt attention on expanded latents (bfloat16): q [total_q, heads, dim + rot_dim] rotated, kv [total_kv, heads * dim | heads *
 * vdim], kr [total_kv, rot_dim] shared by the heads.  A sequence's queries are its last keys; causal.  The result times
 * sigmoid(gate[row, head]) (gate may be null) goes to out [total_q, heads * vdim].  Sizes: fah_latent_prefill_supported. */
int fah_latent_prefill(const void* q, const void* kv, const void* kr, const void* gate, int64_t gate_stride, const int32_t* cu_q,
                       const int32_t* cu_kv, int n_seq, int max_q, int64_t total_q, int64_t total_kv, int heads, int dim, int rot_dim,
                       int vdim, float scale, void* out, int32_t* status, void* stream);
int fah_latent_prefill_supported(int dim, int rot_dim, int vdim, float scale, int dtype);

/* Cached latent rows of every sequence as contiguous rows: c [total_kv, kv_rank], r [total_kv, rot_dim]. */
int fah_latent_gather(const void* pool, int pool_stride, int n_blocks, const int32_t* block_table, int max_blocks, int n_seq,
                      const int32_t* cu_kv, int64_t total_kv, int kv_rank, int rot_dim, void* c, void* r, int32_t* status, int dtype,
                      void* stream);

#ifdef __cplusplus
}
#endif
#endif
