// Prompt attention on expanded latents (see latent_prefill.cu).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace fa {
namespace hybrid {

struct LatentPrefillArgs {
  const void* q;             // bfloat16 [total_q, heads, dim + rot_dim], rotated
  const void* kv;            // bfloat16 [total_kv, heads * dim + heads * vdim]: unrotated keys, then values
  const void* kr;            // bfloat16 [total_kv, rot_dim]: the rotated key part
  const void* gate;          // bfloat16 [total_q, gate_stride] or null
  long long gate_stride;
  const int32_t *cu_q, *cu_kv;   // [n_seq + 1]; a sequence's queries are its last keys
  int n_seq, max_q;
  long long total_q, total_kv;
  int heads, dim, rot_dim, vdim;
  float scale;
  void* out;                 // bfloat16 [total_q, heads * vdim]
  int* status;
};
struct LatentGatherArgs {
  const void* pool;          // T [n_blocks, 16, pool_stride]
  int pool_stride, n_blocks;
  const int32_t* block_table;    // [n_seq, max_blocks]
  int max_blocks, n_seq;
  const int32_t* cu_kv;      // [n_seq + 1]
  long long total_kv;
  int kv_rank, rot_dim;
  void *c, *r;               // T [total_kv, kv_rank], [total_kv, rot_dim]
  int* status;
};

bool latent_prefill_supported(int dim, int rot_dim, int vdim, float scale);
// `encode_fn` is cuTensorMapEncodeTiled.
cudaError_t launch_latent_prefill(const LatentPrefillArgs& a, void* encode_fn, cudaStream_t s);
template <typename T> cudaError_t launch_latent_gather(const LatentGatherArgs& a, cudaStream_t s);

}  // namespace hybrid
}  // namespace fa
