// Preparation of the latent attention's cached rows (see latent_prep.cu).  T: bfloat16 or float activations.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace fa {
namespace hybrid {

struct LatentPrepArgs {
  const void* down;         // T [rows, down_stride]: query latent | key/value latent | shared key part | ...
  long long down_stride;
  int off_q, q_rank, off_kv, kv_rank, off_r, rot_dim;
  const void *wq, *wkv;     // T norm weights
  float eps;
  const float *cos_t, *sin_t;      // [rows, rot_dim / 2]
  void* cq;                 // T [rows, q_rank]
  void* c_out;              // T [rows, kv_rank] or null
  void* r_out;              // T [rows, rot_dim] or null
  void* pool;               // T [n_blocks, 16, pool_stride]
  int pool_stride, n_blocks;
  const int32_t* block_table;      // [n_seq, max_blocks]
  int max_blocks, n_seq;
  const int32_t* tok_seq;   // [rows] sequence of every row
  const int32_t* positions; // [rows] position of every row in its sequence
  long long rows;
  int* status;
};


template <typename T> cudaError_t launch_latent_prep(const LatentPrepArgs& a, cudaStream_t s);
template <typename T> cudaError_t launch_rotate_heads(void* q, const float* cos_t, const float* sin_t, long long rows, int heads,
                                                      int head_stride, int off, int rot_dim, cudaStream_t s);

}  // namespace hybrid
}  // namespace fa
