// Grouped-query attention on paged keys and values inside chunks of the sequence, with a distance bias and an element-wise output
// gate (see kv_attention.cu, kv_decode.cu, kv_prefill.cu).
//
// Position i sees the keys first(i) .. i, first(i) = i - i % chunk (chunk 0: 0); score = scale (q . k) - slope_h (i - j); the output is
// multiplied by sigmoid(gate) column by column.  Pools are [n_blocks, kv_heads, 16, dim] and [n_blocks, kv_heads, 16, vdim].
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace fa {
namespace mixers {

struct Paging {
  int n_blocks;
  const int32_t* block_table;      // [n_seq, max_blocks]
  int max_blocks, n_seq;
  const int32_t* tok_seq;          // [rows] sequence of every row
  const int32_t* positions;        // [rows] position of every row in its sequence
};
struct KvPrepArgs {
  const void* z;             // T [rows, stride]: queries, keys and values at the columns off_q, off_k, off_v
  long long stride;
  int off_q, off_k, off_v, heads, kv_heads, dim, vdim;
  const void *wq, *wk;       // T [heads * dim], [kv_heads * dim]: RMS norms over all heads' columns at once
  float eps;
  const void* v_first;       // T, row stride first_stride: the stored values are (1 - lambda) v + lambda v_first; or null
  long long first_stride;
  float lambda;
  void *q, *k, *v;           // T [rows, ...] contiguous; k and v may be null
  void *k_pool, *v_pool;
  Paging pg;
  long long rows;
  int* status;
};
struct KvAttentionArgs {
  const void* q;             // T [rows, heads, dim]
  const void *k_pool, *v_pool;
  Paging pg;
  const float* slopes;       // [heads]
  const void* gate;          // T [rows, heads * vdim], row stride gate_stride; or null
  long long gate_stride;
  int heads, kv_heads, dim, vdim, chunk;
  float scale;
  void* out;                 // T [rows, heads * vdim], row stride out_stride
  long long out_stride, rows;
  int* status;
  // split kernel
  int splits;
  float* part_o;             // [rows, splits, heads, vdim]
  float* part_ml;            // [rows, splits, heads, 2]
};
struct KvGatherArgs {
  const void *k_pool, *v_pool;
  int n_blocks;
  const int32_t* block_table;
  int max_blocks, n_seq;
  const int32_t *piece_seq, *piece_key0, *cu_kv;   // piece i: keys from position piece_key0[i] on of sequence piece_seq[i]
  int pieces;
  long long total_kv;
  int kv_heads, dim, vdim;
  void *k, *v;               // T [total_kv, kv_heads, dim], [total_kv, kv_heads, vdim]
  int* status;
};
struct KvPrefillArgs {
  const void *q, *k, *v;     // bfloat16 [total_q, heads, dim], [total_kv, kv_heads, dim], [total_kv, kv_heads, vdim]
  const int32_t *cu_q, *cu_kv;   // [n_piece + 1]; a piece's queries are its last keys, causal
  int n_piece, max_q;
  long long total_q, total_kv;
  int heads, kv_heads, dim, vdim;
  float scale;
  const float* slopes;       // [heads]
  const void* gate;          // bfloat16 [total_q, heads * vdim], row stride gate_stride; or null
  long long gate_stride;
  void* out;                 // bfloat16, row stride out_stride
  long long out_stride;
  int* status;
};

template <typename T> cudaError_t launch_kv_prep(const KvPrepArgs& a, cudaStream_t s);
template <typename T> cudaError_t launch_kv_attention(const KvAttentionArgs& a, cudaStream_t s);   // any size, both types
template <typename T> cudaError_t launch_kv_gather(const KvGatherArgs& a, cudaStream_t s);
// Decode steps and short portions (bfloat16).
bool kv_decode_supported(const KvAttentionArgs& a);
int kv_decode_splits(long long rows, int kv_heads, int chunk, int max_blocks, int sm_count);
cudaError_t launch_kv_decode(const KvAttentionArgs& a, cudaStream_t s);
// Prompts (bfloat16).  `encode_fn` is cuTensorMapEncodeTiled.
bool kv_prefill_supported(int heads, int kv_heads, int dim, int vdim, float scale);
cudaError_t launch_kv_prefill(const KvPrefillArgs& a, void* encode_fn, cudaStream_t s);

}  // namespace mixers
}  // namespace fa
