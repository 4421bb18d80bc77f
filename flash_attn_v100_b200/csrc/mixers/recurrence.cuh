// Gated linear recurrences with a matrix state per head (see recurrence.cu, recurrence_gates.cu, recurrence_tc5.cu).
//
//     S_t = e^(la_t) S_(t-1) + b_t k_t v_t^T,      y_t = S_t^T q_t,
// la (at most 0) and b being fp32 numbers per token and head.  Optionally a normaliser n_t = e^(la_t) n_(t-1) + b_t k_t divides:
// y_t = S_t^T q_t / (max(|n_t . q_t|, floor_t) + norm_eps); optionally skip_h v_t is added.  S and n are fp32.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace fa {
namespace mixers {

struct RecurrenceArgs {
  const void* qkv;           // T [total, stride]; per token the queries and keys of heads / kv_rep groups and the heads' values
  long long stride;
  int off_q, off_k, off_v;
  int heads, kv_rep, dk, dv;     // head h has the queries and keys of group h / kv_rep
  float q_scale;
  const float* la;           // [heads, total] log decays
  const float* b;            // [heads, total] weights of the tokens
  const float* floor;        // [heads, total]; null: no normaliser
  const float* n0;           // [n_seq, heads, dk] normaliser before the call
  float* norm;               // [n_slots, 2, heads, dk]: the normaliser after position p is in half p & 1
  float norm_eps;
  const float* skip;         // [heads] or null
  float* state;              // [n_slots, heads, dk, dv]
  int n_slots;
  const int32_t* slots;      // [n_seq] state slot of every sequence
  const int32_t* starts;     // [n_seq] position of the sequence's first token in this call (0: the state starts at zero)
  const int32_t* cu;         // [n_seq + 1] token offsets, or null: sequence i has the one token i
  int n_seq;
  long long total;           // tokens
  void* out;                 // T [total, heads * dv]
  int* status;
  // chunked prompt kernel: a sequence is cut into segments of seg_len tokens that run side by side
  float* seg_state;          // scratch [n_seq, max_segs, heads, dk, dv], max_segs > 1 only
  float* seg_norm;           // scratch [n_seq, max_segs, heads, dk]
  float* seg_log;            // scratch [n_seq, max_segs, heads]: log decay over the segment
  int seg_len, max_segs;
};

// Gates of the exponential-gate memory over prompts: i = cap tanh((z_i + b_i) / cap), f = logsigmoid(cap tanh((z_f + b_f) / cap)), and
// with the running maximum m_t = max(f_t + m_(t-1), i_t): la = f + m_(t-1) - m_t, b = e^(i - m_t), floor = e^(-m_t).
struct MaxGateArgs {
  const void* z;             // T [total, stride]
  long long stride;
  int off_i, off_f, heads;
  const void *bias_i, *bias_f;   // T [heads]
  float cap;
  float* m;                  // [n_slots, 2, heads]: the maximum after position p is in half p & 1
  const float* norm;         // [n_slots, 2, heads, dk], copied to n0 (null: not)
  float* n0;                 // [n_seq, heads, dk]
  int dk, n_slots;
  const int32_t *slots, *starts, *cu;
  int n_seq;
  long long total;
  float *la, *b, *floor;     // [heads, total]
  int* status;
};
// Step sizes of the state-space recurrence: dt = softplus(z + bias), la = -e^(a_log) dt, b = dt.
struct StepGateArgs {
  const void* z;             // T [total, stride], the heads' step logits at column off
  long long stride;
  int off, heads;
  const float *bias, *a_log; // [heads]
  long long total;
  float *la, *b;             // [heads, total]
};
// Causal convolution per channel with SiLU.  The inputs of the last `taps` positions are kept per slot: position p in row p % taps.
struct ConvArgs {
  const void* z;             // T [total, stride], the channels at column off
  long long stride;
  int off, channels, taps;
  const void* w;             // T [taps, channels], the last row is the current token's
  const void* bias;          // T [channels]
  void* ring;                // T [n_slots, taps, channels]
  int n_slots;
  const int32_t *slots, *starts, *cu;   // per sequence; cu null: one token per sequence
  const int32_t *tok_seq, *positions;   // per token
  int n_seq;
  long long total;
  void* out;                 // T [total, channels]
  int* status;
};
// One token per sequence in one kernel: gates (or convolution and step size), state update, output.
struct MaxGateStepArgs {
  RecurrenceArgs r;          // la, b, floor, n0, skip unused
  int off_i, off_f;
  const void *bias_i, *bias_f;
  float cap;
  float* m;                  // [n_slots, 2, heads]
};
struct SsdStepArgs {
  RecurrenceArgs r;          // qkv is the projection: off_v, off_k, off_q are the columns of x, B and C (adjacent, in this order)
  int off_dt;
  const float *dt_bias, *a_log;
  const void *conv_w, *conv_b;   // as ConvArgs
  void* ring;
  int taps;
};

// Token by token: any size, both types.
template <typename T> cudaError_t launch_recurrence_scan(const RecurrenceArgs& a, cudaStream_t s);
template <typename T> cudaError_t launch_max_gates(const MaxGateArgs& a, cudaStream_t s);
template <typename T> cudaError_t launch_step_gates(const StepGateArgs& a, cudaStream_t s);
template <typename T> cudaError_t launch_conv_silu(const ConvArgs& a, cudaStream_t s);
// One token per sequence; dv a multiple of 4 and at most 1024, dk at most 1024.
bool recurrence_step_supported(const RecurrenceArgs& a);
template <typename T> cudaError_t launch_max_gate_step(const MaxGateStepArgs& a, int sm_count, cudaStream_t s);
template <typename T> cudaError_t launch_ssd_step(const SsdStepArgs& a, int sm_count, cudaStream_t s);

// Prompts in chunks on the tensor cores (bfloat16; dk <= 128, dk and dv multiples of 8).  `encode_fn` is cuTensorMapEncodeTiled.
int recurrence_segments(int n_seq, int heads, int kv_rep, int dk, int dv, int max_len, int sm_count, int* seg_len);
bool recurrence_tc5_supported(const RecurrenceArgs& a);
cudaError_t launch_recurrence_tc5(const RecurrenceArgs& a, void* encode_fn, cudaStream_t s);

}  // namespace mixers
}  // namespace fa
