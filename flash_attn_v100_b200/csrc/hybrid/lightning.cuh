// Decayed linear attention (see lightning.cu and lightning_chunk.cu).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace fa {
namespace hybrid {

struct LightningArgs {
  const void* qkv;           // T [tokens, stride]; per token the H x dk queries, H x dk keys and H x dv values
  long long stride;
  int off_q, off_k, off_v;
  int heads, dk, dv;
  const float* decay;        // [heads]
  float* state;              // [n_slots, heads, dk, dv]
  int n_slots;
  const int32_t* slots;      // [n_seq] state slot of every sequence
  const int32_t* starts;     // [n_seq] position of the sequence's first token in this call (0: the state starts at zero)
  const int32_t* cu;         // [n_seq + 1] token offsets, or null: sequence i has the one token i
  int n_seq;
  long long total;           // tokens
  void* out;                 // T [tokens, heads * dv]
  int* status;
  // chunked prompt kernel: a sequence is cut into segments of seg_len tokens that run side by side
  float* seg_state;          // scratch [n_seq, max_segs, heads, dk, dv] (max_segs > 1 only)
  int seg_len, max_segs;
};

// Token-by-token kernel: any size, both types; prompts and decode steps.
template <typename T> cudaError_t launch_lightning_scan(const LightningArgs& a, cudaStream_t s);
// One token per sequence; dv a multiple of 4 and at most 1024.
template <typename T> cudaError_t launch_lightning_decode(const LightningArgs& a, int sm_count, cudaStream_t s);
bool lightning_decode_supported(const LightningArgs& a);


// Prompts in chunks on the tensor cores (bfloat16; dk <= 128, dk and dv multiples of 8).
// Segments per sequence and their length (a multiple of the chunk) for the longest sequence of a call.
int lightning_segments(int n_seq, int heads, int dk, int dv, int max_len, int sm_count, int* seg_len);
bool lightning_chunk_supported(const LightningArgs& a);
cudaError_t launch_lightning_chunk(const LightningArgs& a, cudaStream_t s);   // dk, dv <= 64, mma.sync
cudaError_t launch_lightning_tc5(const LightningArgs& a, cudaStream_t s);     // larger heads, tcgen05
// Turns what every segment adds to the state into the state at the start of every segment.
cudaError_t launch_lightning_segment_scan(const LightningArgs& a, cudaStream_t s);

}  // namespace hybrid
}  // namespace fa
