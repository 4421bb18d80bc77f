// Row-wise operators of the hybrid decoders (see row_ops.cu).  T: bfloat16 or float activations.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace fa {
namespace hybrid {

struct ResidualNormArgs {
  float* x;                 // [rows, cols] residual, updated in place
  const void* delta;        // T [rows, cols] or null
  const void* delta_w;      // T [cols]: delta is RMS-normed with this weight before it is added; or null
  const void* embed;        // T [vocab, cols] or null
  const int64_t* tokens;    // [rows] rows of embed
  int embed_mode;           // 0: unused, 1: x += embed[token], 2: x = embed[token] * embed_scale + the further tables' rows
  const void* w;            // T [cols] or null: out is the plain x
  void* out;                // T [rows, cols] or null
  long long rows;
  int cols, vocab;
  float eps;
  const void* w2;           // T [cols]: a second norm of the same x
  void* out2;               // T [rows, cols] or null
  float embed_scale;
  const void* more[2];      // T [more_n, cols] or null (embed_mode 2)
  const int32_t* more_rows[2];   // [rows] rows of the further tables
  int more_n[2];
};
struct GatedNormArgs {
  const void* o;            // T [rows, cols]
  const void* g;            // T, row stride g_stride
  long long g_stride;
  const void* w;            // T [cols]
  void* out;                // T, row stride out_stride
  long long out_stride;
  long long rows;
  int cols, group;          // the norm is taken over `group` columns at a time
  float eps;
  int silu_first;           // 1: rmsnorm(o * silu(g)) * w, 0: rmsnorm(o) * w * sigmoid(g)
};

template <typename T> cudaError_t launch_residual_norm(const ResidualNormArgs& a, cudaStream_t s);
template <typename T> cudaError_t launch_gated_norm(const GatedNormArgs& a, cudaStream_t s);
template <typename T> cudaError_t launch_gelu(const void* z, long long z_stride, void* out, long long out_stride, long long rows, int n,
                                              cudaStream_t s);
template <typename T> cudaError_t launch_clamped_glu(const void* gu, void* out, long long rows, int n, float limit, float alpha,
                                                     float shift, cudaStream_t s);
template <typename T> cudaError_t launch_side_gate(const void* z, const void* side, const int64_t* tokens, int vocab,
                                                   long long side_stride, int off, void* out, long long rows, int n, cudaStream_t s);
cudaError_t launch_bigram_rows(const int64_t* tokens, const int32_t* cu, const int32_t* starts, const int32_t* slots, int32_t* last, int n_slots,
                               int n_seq, long long total, long long buckets, long long mul_prev, long long mul_cur, int32_t* out, int* status,
                               cudaStream_t s);

}  // namespace hybrid
}  // namespace fa
