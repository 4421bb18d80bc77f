// Gated linear recurrences, sm_100a: the token-by-token kernel for any size, and the decode steps, which compute the gates (and the
// short convolution) of their token themselves.
//
// The state S [dk, dv] of every head is fp32 and lives in a slot of the cache between calls.  A sequence whose first token is at
// position 0 starts from zero whatever its slot holds.  The normaliser and the running maximum are kept twice, by the parity of the
// position, so that the CTAs of one head can read the old one while one of them writes the new one.
#include "../hybrid/hybrid_common.cuh"
#include "recurrence.cuh"

namespace fa {
namespace mixers {

using hybrid::bf16;
using hybrid::block_sum;
using hybrid::from_f;
using hybrid::sigmoid_f;
using hybrid::silu_f;
using hybrid::to_f;
using hybrid::warp_sum;

namespace {

constexpr int kCols = 32;      // value columns per CTA of the scan kernel
constexpr int kRowGroups = 8;

template <typename T>
__global__ void __launch_bounds__(kCols * kRowGroups) recurrence_scan_kernel(const RecurrenceArgs a) {
  extern __shared__ float sm[];
  float* S = sm;                          // [dk][kCols]
  float* sq = S + a.dk * kCols;           // [dk]
  float* sk = sq + a.dk;                  // [dk]
  float* sn = sk + a.dk;                  // [dk]
  float* red = sn + a.dk;                 // [kRowGroups][kCols]
  float* redn = red + kRowGroups * kCols; // [kRowGroups]
  const int seq = blockIdx.x, head = blockIdx.y, c0 = blockIdx.z * kCols;
  const int lane = threadIdx.x & 31, rg = threadIdx.x >> 5;
  const int col = c0 + lane, grp = head / a.kv_rep;
  const bool live = col < a.dv;
  long long t0 = seq, t1 = seq + 1;
  if (a.cu != nullptr) {
    t0 = a.cu[seq];
    t1 = a.cu[seq + 1];
  }
  if (t0 < 0) t0 = 0;
  if (t1 > a.total) t1 = a.total;
  const int n = t1 > t0 ? (int)(t1 - t0) : 0;
  if (n == 0) return;
  const int slot = a.slots[seq];
  float* state = nullptr;
  if (slot >= 0 && slot < a.n_slots) state = a.state + ((long long)slot * a.heads + head) * a.dk * a.dv;
  else if (threadIdx.x == 0) atomicOr(a.status, 2);
  const bool fresh = a.starts[seq] == 0;
  for (int r = rg; r < a.dk; r += kRowGroups)
    S[r * kCols + lane] = (!fresh && live && state) ? state[(long long)r * a.dv + col] : 0.f;
  const bool normed = a.floor != nullptr;
  if (normed)
    for (int i = threadIdx.x; i < a.dk; i += blockDim.x) sn[i] = a.n0[((long long)seq * a.heads + head) * a.dk + i];
  const T* base = static_cast<const T*>(a.qkv);
  T* out = static_cast<T*>(a.out);
  const float skip = a.skip != nullptr ? a.skip[head] : 0.f;
  for (int t = 0; t < n; ++t) {
    const T* row = base + (t0 + t) * a.stride;
    const long long ht = (long long)head * a.total + t0 + t;
    const float d = expf(a.la[ht]), w = a.b[ht];
    __syncthreads();
    float nq = 0.f;
    for (int i = threadIdx.x; i < a.dk; i += blockDim.x) {
      const float q = to_f(row[a.off_q + grp * a.dk + i]) * a.q_scale, k = to_f(row[a.off_k + grp * a.dk + i]);
      sq[i] = q;
      sk[i] = k;
      if (normed) {
        const float v = d * sn[i] + w * k;
        sn[i] = v;
        nq += v * q;
      }
    }
    if (normed) {
      nq = warp_sum(nq);
      if (lane == 0) redn[rg] = nq;
    }
    const float v = live ? to_f(row[a.off_v + head * a.dv + col]) : 0.f;
    const float wv = w * v;
    __syncthreads();
    float o = 0.f;
    for (int r = rg; r < a.dk; r += kRowGroups) {
      const float s = d * S[r * kCols + lane] + sk[r] * wv;
      S[r * kCols + lane] = s;
      o += sq[r] * s;
    }
    red[rg * kCols + lane] = o;
    __syncthreads();
    if (rg == 0 && live) {
#pragma unroll
      for (int i = 1; i < kRowGroups; ++i) o += red[i * kCols + lane];
      if (normed) {
        float den = 0.f;
#pragma unroll
        for (int i = 0; i < kRowGroups; ++i) den += redn[i];
        o /= fmaxf(fabsf(den), a.floor[ht]) + a.norm_eps;
      }
      out[(t0 + t) * (long long)a.heads * a.dv + (long long)head * a.dv + col] = from_f<T>(o + skip * v);
    }
  }
  if (state && live)
    for (int r = rg; r < a.dk; r += kRowGroups) state[(long long)r * a.dv + col] = S[r * kCols + lane];
  if (normed && state && blockIdx.z == 0) {
    const int half = (a.starts[seq] + n - 1) & 1;
    for (int i = threadIdx.x; i < a.dk; i += blockDim.x)
      a.norm[(((long long)slot * 2 + half) * a.heads + head) * a.dk + i] = sn[i];
  }
}

enum { kMaxGate = 0, kSsd = 1 };
template <int KIND> struct StepArgs;
template <> struct StepArgs<kMaxGate> { using type = MaxGateStepArgs; };
template <> struct StepArgs<kSsd> { using type = SsdStepArgs; };

// CTA = (sequence, head, range of value columns); a thread owns four columns of every n_rg-th state row, so the state is read and
// written once with 16-byte accesses.  The first rows are on their way while the gates are computed.
template <typename T, int KIND>
__global__ void __launch_bounds__(256) recurrence_step_kernel(const typename StepArgs<KIND>::type p, const int cols) {
  extern __shared__ float sm[];
  const RecurrenceArgs& a = p.r;
  float* sq = sm;                         // [dk]
  float* sk = sq + a.dk;                  // [dk]
  float* red = sk + a.dk;                 // [n_rg][cols]
  __shared__ float warp_red[8];
  const int seq = blockIdx.x, head = blockIdx.y, c0 = blockIdx.z * cols, grp = head / a.kv_rep;
  const int my_cols = min(cols, a.dv - c0);
  const int n4 = cols / 4, n_rg = blockDim.x / n4;
  const int cg = threadIdx.x % n4, rg = threadIdx.x / n4;
  const int slot = a.slots[seq];
  if (slot < 0 || slot >= a.n_slots) {    // (uniform over the CTA)
    if (threadIdx.x == 0) atomicOr(a.status, 2);
    return;
  }
  const int pos = a.starts[seq];
  const bool fresh = pos == 0;
  float* state = a.state + ((long long)slot * a.heads + head) * a.dk * a.dv;
  const bool live = rg < n_rg && cg * 4 < my_cols;
  float* sp = state + c0 + cg * 4;
  constexpr int U = 8;
  float4 s0[U];
  const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int u = 0; u < U; ++u)
    s0[u] = live && !fresh && rg + u * n_rg < a.dk ? *reinterpret_cast<const float4*>(sp + (long long)(rg + u * n_rg) * a.dv) : zero4;

  const T* row = static_cast<const T*>(a.qkv) + (long long)seq * a.stride;
  float v[4] = {0.f, 0.f, 0.f, 0.f};
  float d, w, scale_out = 1.f, skip = 0.f;
  if constexpr (KIND == kMaxGate) {
    const float zi = to_f(row[p.off_i + head]) + to_f(static_cast<const T*>(p.bias_i)[head]);
    const float zf = to_f(row[p.off_f + head]) + to_f(static_cast<const T*>(p.bias_f)[head]);
    const float gi = p.cap * tanhf(zi / p.cap), gf = p.cap * tanhf(zf / p.cap);
    const float f = gf < 0.f ? gf - log1pf(expf(gf)) : -log1pf(expf(-gf));
    const float m_old = fresh ? 0.f : p.m[((long long)slot * 2 + ((pos - 1) & 1)) * a.heads + head];
    const float m = fmaxf(f + m_old, gi);
    d = expf(f + m_old - m);
    w = expf(gi - m);
    float nq = 0.f;
    const float* n_old = a.norm + (((long long)slot * 2 + ((pos - 1) & 1)) * a.heads + head) * a.dk;
    float* n_new = a.norm + (((long long)slot * 2 + (pos & 1)) * a.heads + head) * a.dk;
    for (int i = threadIdx.x; i < a.dk; i += blockDim.x) {
      const float q = to_f(row[a.off_q + grp * a.dk + i]) * a.q_scale, k = to_f(row[a.off_k + grp * a.dk + i]);
      sq[i] = q;
      sk[i] = k;
      const float n = (fresh ? 0.f : d * n_old[i]) + w * k;
      if (blockIdx.z == 0) n_new[i] = n;
      nq += n * q;
    }
    if (live) {
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] = to_f(row[a.off_v + head * a.dv + c0 + cg * 4 + j]);
    }
    nq = block_sum(nq, warp_red);
    scale_out = 1.f / (fmaxf(fabsf(nq), expf(-m)) + a.norm_eps);
    if (blockIdx.z == 0 && threadIdx.x == 0) p.m[((long long)slot * 2 + (pos & 1)) * a.heads + head] = m;
  } else {
    const float z = to_f(row[p.off_dt + head]) + p.dt_bias[head];
    const float dt = z > 0.f ? z + log1pf(expf(-z)) : log1pf(expf(z));
    d = expf(-expf(p.a_log[head]) * dt);
    w = dt;
    skip = a.skip[head];
    // channel c (counted from the column of x) through the convolution; the current input is kept for the next positions
    const int taps = p.taps, channels = a.off_q + (a.heads / a.kv_rep) * a.dk - a.off_v;
    T* ring = static_cast<T*>(p.ring) + (long long)slot * taps * channels;
    auto conv = [&](int c, bool keep) {
      const T* wt = static_cast<const T*>(p.conv_w);
      const T in = row[a.off_v + c];
      float acc = to_f(static_cast<const T*>(p.conv_b)[c]) + to_f(wt[(taps - 1) * channels + c]) * to_f(in);
      for (int k = 1; k < taps && k <= pos; ++k)
        acc += to_f(wt[(taps - 1 - k) * channels + c]) * to_f(ring[(long long)((pos - k) % taps) * channels + c]);
      if (keep) ring[(long long)(pos % taps) * channels + c] = in;
      return to_f(from_f<T>(silu_f(acc)));
    };
    const bool first = blockIdx.z == 0 && head % a.kv_rep == 0;
    for (int i = threadIdx.x; i < 2 * a.dk; i += blockDim.x) {
      const int j = i < a.dk ? i : i - a.dk;
      if (i < a.dk) sq[j] = conv(a.off_q - a.off_v + grp * a.dk + j, first);
      else sk[j] = conv(a.off_k - a.off_v + grp * a.dk + j, first);
    }
    // my value columns by way of shared memory: every channel is convolved (and kept) by one thread
    for (int c = threadIdx.x; c < my_cols; c += blockDim.x) red[c] = conv(head * a.dv + c0 + c, true);
    __syncthreads();
    if (live) {
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] = red[cg * 4 + j];
    }
  }
  __syncthreads();
  float wv[4], o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int j = 0; j < 4; ++j) wv[j] = w * v[j];
  if (live) {
    for (int r = rg; r < a.dk; r += U * n_rg) {
      float4 s[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (r == rg) s[u] = s0[u];
        else s[u] = !fresh && r + u * n_rg < a.dk ? *reinterpret_cast<const float4*>(sp + (long long)(r + u * n_rg) * a.dv) : zero4;
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (r + u * n_rg >= a.dk) break;
        const float k = sk[r + u * n_rg], q = sq[r + u * n_rg];
        s[u].x = d * s[u].x + k * wv[0]; s[u].y = d * s[u].y + k * wv[1];
        s[u].z = d * s[u].z + k * wv[2]; s[u].w = d * s[u].w + k * wv[3];
        *reinterpret_cast<float4*>(sp + (long long)(r + u * n_rg) * a.dv) = s[u];
        o[0] += q * s[u].x; o[1] += q * s[u].y; o[2] += q * s[u].z; o[3] += q * s[u].w;
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) red[rg * cols + cg * 4 + j] = o[j] * scale_out + (rg == 0 ? skip * v[j] : 0.f);
  } else if (rg < n_rg) {
#pragma unroll
    for (int j = 0; j < 4; ++j) red[rg * cols + cg * 4 + j] = 0.f;
  }
  __syncthreads();
  T* out = static_cast<T*>(a.out) + (long long)seq * a.heads * a.dv + (long long)head * a.dv + c0;
  for (int c = threadIdx.x; c < my_cols; c += blockDim.x) {
    float acc = 0.f;
    for (int i = 0; i < n_rg; ++i) acc += red[i * cols + c];
    out[c] = from_f<T>(acc);
  }
}

template <typename T, int KIND>
cudaError_t launch_step(const typename StepArgs<KIND>::type& p, int sm_count, cudaStream_t s) {
  const RecurrenceArgs& a = p.r;
  if (a.n_seq == 0) return cudaSuccess;
  // value columns per CTA: the whole head, or a part of it while that leaves SMs without work
  int cols = (a.dv + 31) / 32 * 32;
  while (cols > 32 && (long long)a.n_seq * a.heads * ((a.dv + cols - 1) / cols) < 2ll * sm_count) cols = (cols / 2 + 31) / 32 * 32;
  const int n_rg = 256 / (cols / 4);
  const size_t smem = ((size_t)2 * a.dk + (size_t)n_rg * cols) * sizeof(float);
  dim3 grid((unsigned)a.n_seq, (unsigned)a.heads, (unsigned)((a.dv + cols - 1) / cols));
  recurrence_step_kernel<T, KIND><<<grid, 256, smem, s>>>(p, cols);
  return cudaGetLastError();
}

}  // namespace

template <typename T>
cudaError_t launch_recurrence_scan(const RecurrenceArgs& a, cudaStream_t s) {
  if (a.n_seq == 0) return cudaSuccess;
  const size_t smem = ((size_t)a.dk * (kCols + 3) + kRowGroups * (kCols + 1)) * sizeof(float);
  cudaError_t e = cudaFuncSetAttribute(recurrence_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  dim3 grid((unsigned)a.n_seq, (unsigned)a.heads, (unsigned)((a.dv + kCols - 1) / kCols));
  recurrence_scan_kernel<T><<<grid, kCols * kRowGroups, smem, s>>>(a);
  return cudaGetLastError();
}

bool recurrence_step_supported(const RecurrenceArgs& a) {
  return a.cu == nullptr && a.dv % 4 == 0 && a.dv <= 1024 && a.dk <= 1024 && (reinterpret_cast<uintptr_t>(a.state) & 15) == 0;
}

template <typename T>
cudaError_t launch_max_gate_step(const MaxGateStepArgs& a, int sm_count, cudaStream_t s) { return launch_step<T, kMaxGate>(a, sm_count, s); }
template <typename T>
cudaError_t launch_ssd_step(const SsdStepArgs& a, int sm_count, cudaStream_t s) { return launch_step<T, kSsd>(a, sm_count, s); }

#define FA_RECURRENCE(T)                                                           \
  template cudaError_t launch_recurrence_scan<T>(const RecurrenceArgs&, cudaStream_t); \
  template cudaError_t launch_max_gate_step<T>(const MaxGateStepArgs&, int, cudaStream_t); \
  template cudaError_t launch_ssd_step<T>(const SsdStepArgs&, int, cudaStream_t);
FA_RECURRENCE(bf16)
FA_RECURRENCE(float)

}  // namespace mixers
}  // namespace fa
