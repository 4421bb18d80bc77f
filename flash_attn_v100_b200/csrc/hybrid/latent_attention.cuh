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
  // split-KV decode only
  int n_split;
  float* part_o;             // [n_split, rows, heads, kv_rank]
  float* part_ml;            // [n_split, rows, heads, 2] (maximum in log2 units, sum)
};

// One CTA per (row, head): any size, both types.
template <typename T> cudaError_t launch_latent_attention(const LatentAttentionArgs& a, cudaStream_t s);

}  // namespace hybrid
}  // namespace fa
