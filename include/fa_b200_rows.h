/* C ABI of the row-wise operators between the matrix products of the hybrid decoders (libfa_b200_rows.so, sm_100a).
 *
 * Conventions: device pointers on the current device; every call is asynchronous on `stream` (a cudaStream_t);
 * nothing is allocated.  `dtype` is the type of activations and weights: FAR_F32 or FAR_BF16; the residual stream is
 * always fp32.  `status` is one int32 in device memory that the caller has set to zero: a kernel that meets a state slot
 * outside the cache sets bit 1 in it and skips the access.  Return value: 0, or a negative code with a text in
 * far_last_error(). */
#ifndef FA_B200_ROWS_H
#define FA_B200_ROWS_H
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

enum { FAR_F32 = 0, FAR_BF16 = 1 };
enum { FAR_OK = 0, FAR_ERR_INVALID_ARGUMENT = -1, FAR_ERR_UNSUPPORTED = -2, FAR_ERR_CUDA = -4 };

const char* far_last_error(void);

/* x [rows, cols] fp32: embed_mode 1 adds embed[token], 2 sets x to embed[token] * embed_scale plus row more_rows[k][r] of every
 * further table more[k] [more_n[k], cols]; then delta [rows, cols] is added, RMS-normed with weight delta_w first if that is
 * given.  out [rows, cols] = rmsnorm(x) * w, or x itself if w is null; out may be null.  out2 = rmsnorm(x) * w2 where w2 is
 * given.  Unused pointers are null, an unused embed_scale is 1. */
typedef struct {
  float* x;
  const void *delta, *delta_w, *embed;
  const int64_t* tokens;
  int32_t embed_mode, vocab;
  float embed_scale, eps;
  const void* more[2];
  const int32_t* more_rows[2];
  int32_t more_n[2];
  const void *w, *w2;
  void *out, *out2;
  int64_t rows;
  int32_t cols, dtype;
} FarResidualNorm;
int far_residual_norm(const FarResidualNorm* args, void* stream);

/* The norm is taken over every `group` columns of a row (cols: the whole row).  out = rmsnorm(o [rows, cols]) * w * sigmoid(g), or
 * with silu_first rmsnorm(o * silu(g)) * w; g and out have the row strides g_stride and out_stride. */
int far_gated_norm(const void* o, const void* g, int64_t g_stride, const void* w, void* out, int64_t out_stride, int64_t rows, int cols, int group,
                   int silu_first, float eps, int dtype, void* stream);

/* out [rows, n] = gelu_tanh(z [rows, n]), with the row strides out_stride and z_stride. */
int far_gelu(const void* z, int64_t z_stride, void* out, int64_t out_stride, int64_t rows, int n, int dtype, void* stream);

/* out[t] = (previous token * mul_prev + tokens[t] * mul_cur) mod buckets, or `buckets` for the first token of a sequence (starts 0).
 * The token before a call is taken from last[slots[seq]], where the call's last token is left.  cu_seqlens null: one token
 * per sequence. */
int far_bigram_rows(const int64_t* tokens, const int32_t* cu_seqlens, const int32_t* starts, const int32_t* slots, int32_t* last, int n_slots, int n_seq,
                    int64_t total, int64_t buckets, int64_t mul_prev, int64_t mul_cur, int32_t* out, int32_t* status, void* stream);

/* gu [rows, 2n]: out [rows, n] = g * sigmoid(alpha * g) * (u + shift), g = min(gu[:n], limit), u = clamp(gu[n:], -limit, limit). */
int far_clamped_glu(const void* gu, void* out, int64_t rows, int n, float limit, float alpha, float shift, int dtype,
                    void* stream);

/* out [rows, n] = gelu_tanh(z [rows, n]) * side[token, off : off + n], side with row stride side_stride. */
int far_side_gate(const void* z, const void* side, const int64_t* tokens, int vocab, int64_t side_stride, int off, void* out,
                  int64_t rows, int n, int dtype, void* stream);

#ifdef __cplusplus
}
#endif
#endif
