// Attention over the cached latent rows (see latent_attention.cu, latent_decode.cu).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace fa {
namespace hybrid {

struct LatentAttentionArgs {
  const void* q_abs;         // T [rows, heads, kv_rank]: unrotated query part, multiplied into the latent space
  const void* q;             // T [rows, heads, q_stride]: the rotated query part before its rotation, at column q_off
  int q_stride, q_off;
  const float *cos_t, *sin_t;    // [rows, rot_dim / 2]
  const void* pool;          // T [n_blocks, 16, pool_stride]: latent | rotated key part
  int pool_stride, n_blocks;
  const int32_t* block_table;    // [n_seq, max_blocks]
  int max_blocks, n_seq;
  const int32_t* tok_seq;    // [rows]
  const int32_t* positions;  // [rows]: the row sees the keys 0 .. position
  const void* gate;          // T [rows, gate_stride]: head h's output is multiplied by sigmoid(gate[h]); or null
  long long gate_stride;
  int heads, kv_rank, rot_dim;
  float scale;
  void* out;                 // T [rows, heads, kv_rank]
  long long rows;
  int* status;
  // tensor-core kernel: work is cut into equal runs of key tiles, one per CTA and head block
  int n_cta;
  float* part_o;             // [n_cta, 2, heads, kv_rank] unnormalised sums of the rows that are cut
  float* part_ml;            // [n_cta, 2, heads, 2]: their maxima (log2 units) and weights
  int32_t* row_tiles;        // [rows + 1] prefix sums of the rows' key tiles, written by the kernel for the merge
};

// One CTA per (row, head): any size, both types.
template <typename T> cudaError_t launch_latent_attention(const LatentAttentionArgs& a, cudaStream_t s);


// Tensor cores (bfloat16; kv_rank + rot_dim <= 576, both multiples of 8).
bool latent_decode_supported(const LatentAttentionArgs& a);
int latent_decode_ctas(int heads, int sm_count);   // per head block
cudaError_t launch_latent_decode(const LatentAttentionArgs& a, void* encode_fn, cudaStream_t s);   // cuTensorMapEncodeTiled

}  // namespace hybrid
}  // namespace fa
