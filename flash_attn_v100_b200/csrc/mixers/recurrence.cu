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
using hybrid::from_f;
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

constexpr int kMaxBlockHeads = 8;

// CTA = (sequence, block of `hb` heads, range of value columns): the heads' tokens are prepared together (of the state-space recurrence
// only heads of one group, which share keys and queries), then their states go by one after the other, the next rows on their way while
// the current ones are worked on.  A thread owns four columns of every n_rg-th state row, so the state is read and written once with
// 16-byte accesses.  TAPS: of the convolution (0: any number).
template <typename T, int KIND, int TAPS>
__global__ void __launch_bounds__(256) recurrence_step_kernel(const typename StepArgs<KIND>::type p, const int cols, const int hb) {
  extern __shared__ float sm[];
  const RecurrenceArgs& a = p.r;
  constexpr bool OWN = KIND == kMaxGate;  // every head has keys and queries of its own
  const int dk = a.dk, dkp = (dk + 3) & ~3, n4 = cols / 4, n_rg = 256 / n4;
  float* sq = sm;                         // [hb or 1][dkp]
  float* sk = sq + (OWN ? hb : 1) * dkp;  // [hb or 1][dkp]
  float* sv = sk + (OWN ? hb : 1) * dkp;  // [hb][cols]
  float* red = sv + hb * cols;            // [2][n_rg][cols]
  __shared__ float s_decay[kMaxBlockHeads], s_weight[kMaxBlockHeads], s_scale[kMaxBlockHeads], s_skip[kMaxBlockHeads];
  const int seq = blockIdx.x, head0 = blockIdx.y * hb, c0 = blockIdx.z * cols, grp = head0 / a.kv_rep;
  const int my_cols = min(cols, a.dv - c0);
  const int tid = threadIdx.x, cg = tid % n4, rg = tid / n4;
  const int slot = a.slots[seq];
  if (slot < 0 || slot >= a.n_slots) {    // (uniform over the CTA)
    if (tid == 0) atomicOr(a.status, 2);
    return;
  }
  const int pos = a.starts[seq];
  const bool fresh = pos == 0;
  const long long hs = (long long)dk * a.dv;
  const bool live = rg < n_rg && cg * 4 < my_cols;
  float* sp = a.state + ((long long)slot * a.heads + head0) * hs + c0 + cg * 4;
  constexpr int U = 8;
  const int batches = (dk + U * n_rg - 1) / (U * n_rg), steps = hb * batches;
  float4 s[U], nx[U];
  const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
  auto fetch = [&](int step, float4 (&v)[U]) {
    const int hh = step / batches, r0 = (step - hh * batches) * U * n_rg + rg;
    const float* q = sp + hh * hs;
#pragma unroll
    for (int u = 0; u < U; ++u)
      v[u] = live && !fresh && r0 + u * n_rg < dk ? *reinterpret_cast<const float4*>(q + (long long)(r0 + u * n_rg) * a.dv) : zero4;
  };
  fetch(0, s);

  // ---- the heads' tokens ------------------------------------------------------------------------------
  const T* row = static_cast<const T*>(a.qkv) + (long long)seq * a.stride;
  if constexpr (KIND == kMaxGate) {
    float m = 0.f;
    if (tid < hb) {
      const int head = head0 + tid;
      const float zi = to_f(row[p.off_i + head]) + to_f(static_cast<const T*>(p.bias_i)[head]);
      const float zf = to_f(row[p.off_f + head]) + to_f(static_cast<const T*>(p.bias_f)[head]);
      const float gi = p.cap * tanhf(zi / p.cap), gf = p.cap * tanhf(zf / p.cap);
      const float f = gf < 0.f ? gf - log1pf(expf(gf)) : -log1pf(expf(-gf));
      const float m_old = fresh ? 0.f : p.m[((long long)slot * 2 + ((pos - 1) & 1)) * a.heads + head];
      m = fmaxf(f + m_old, gi);
      s_decay[tid] = expf(f + m_old - m);
      s_weight[tid] = expf(gi - m);
      s_scale[tid] = expf(-m);
      s_skip[tid] = 0.f;
      if (blockIdx.z == 0) p.m[((long long)slot * 2 + (pos & 1)) * a.heads + head] = m;
    }
    for (int i = tid; i < hb * dk; i += 256) {
      const int hh = i / dk, j = hh * dkp + i - hh * dk;
      sq[j] = to_f(row[a.off_q + head0 * dk + i]) * a.q_scale;
      sk[j] = to_f(row[a.off_k + head0 * dk + i]);
    }
    for (int i = tid; i < hb * my_cols; i += 256) {
      const int hh = i / my_cols, c = i - hh * my_cols;
      sv[hh * cols + c] = to_f(row[a.off_v + (head0 + hh) * a.dv + c0 + c]);
    }
    __syncthreads();
    // a warp per head: the normaliser
    const float* n_old = a.norm + (((long long)slot * 2 + ((pos - 1) & 1)) * a.heads + head0) * dk;
    float* n_new = a.norm + (((long long)slot * 2 + (pos & 1)) * a.heads + head0) * dk;
    for (int hh = tid >> 5; hh < hb; hh += 8) {
      const float d = s_decay[hh], w = s_weight[hh];
      float nq = 0.f;
      for (int i = tid & 31; i < dk; i += 32) {
        const float n = (fresh ? 0.f : d * n_old[hh * dk + i]) + w * sk[hh * dkp + i];
        if (blockIdx.z == 0) n_new[hh * dk + i] = n;
        nq += n * sq[hh * dkp + i];
      }
      nq = warp_sum(nq);
      if ((tid & 31) == 0) s_scale[hh] = 1.f / (fmaxf(fabsf(nq), s_scale[hh]) + a.norm_eps);
    }
  } else {
    if (tid < hb) {
      const int head = head0 + tid;
      const float z = to_f(row[p.off_dt + head]) + p.dt_bias[head];
      const float dt = z > 0.f ? z + log1pf(expf(-z)) : log1pf(expf(z));
      s_decay[tid] = expf(-expf(p.a_log[head]) * dt);
      s_weight[tid] = dt;
      s_scale[tid] = 1.f;
      s_skip[tid] = a.skip[head];
    }
    // channel c (counted from the column of the values) through the convolution; the current input is kept for the next positions
    const int taps = TAPS > 0 ? TAPS : p.taps, channels = a.off_q + (a.heads / a.kv_rep) * dk - a.off_v;
    T* ring = static_cast<T*>(p.ring) + (long long)slot * taps * channels;
    const T* wt = static_cast<const T*>(p.conv_w);
    const int at = pos % taps;
    auto conv = [&](int c, bool keep) {
      const T in = row[a.off_v + c];
      float acc = to_f(static_cast<const T*>(p.conv_b)[c]) + to_f(wt[(taps - 1) * channels + c]) * to_f(in);
      if constexpr (TAPS > 0) {
        float old[TAPS > 1 ? TAPS - 1 : 1], w[TAPS > 1 ? TAPS - 1 : 1];
#pragma unroll
        for (int k = 1; k < TAPS; ++k) {
          old[k - 1] = k <= pos ? to_f(ring[(at >= k ? at - k : at - k + TAPS) * channels + c]) : 0.f;
          w[k - 1] = to_f(wt[(TAPS - 1 - k) * channels + c]);
        }
#pragma unroll
        for (int k = 1; k < TAPS; ++k) acc += w[k - 1] * old[k - 1];
      } else {
        for (int k = 1; k < taps && k <= pos; ++k)
          acc += to_f(wt[(taps - 1 - k) * channels + c]) * to_f(ring[(long long)((pos - k) % taps) * channels + c]);
      }
      if (keep) ring[(long long)at * channels + c] = in;
      return to_f(from_f<T>(silu_f(acc)));
    };
    const bool first = blockIdx.z == 0 && head0 % a.kv_rep == 0;        // every channel is kept by one CTA
    const int n = 2 * dk + hb * my_cols;
    for (int i = tid; i < n; i += 256) {
      if (i < dk) {
        sq[i] = conv(a.off_q - a.off_v + grp * dk + i, first);
      } else if (i < 2 * dk) {
        sk[i - dk] = conv(a.off_k - a.off_v + grp * dk + i - dk, first);
      } else {
        const int hh = (i - 2 * dk) / my_cols, c = i - 2 * dk - hh * my_cols;
        sv[hh * cols + c] = conv((head0 + hh) * a.dv + c0 + c, true);
      }
    }
  }
  __syncthreads();

  // ---- the heads' states ------------------------------------------------------------------------------
  T* out = static_cast<T*>(a.out) + (long long)seq * a.heads * a.dv + (long long)head0 * a.dv + c0;
  float o[4] = {0.f, 0.f, 0.f, 0.f};
  for (int step = 0; step < steps; ++step) {
    const int hh = step / batches, bt = step - hh * batches;
    if (step + 1 < steps) fetch(step + 1, nx);
    const float d = s_decay[hh], w = s_weight[hh];
    const float *q = sq + (OWN ? hh * dkp : 0), *k = sk + (OWN ? hh * dkp : 0);
    if (live) {
      const float4 v = *reinterpret_cast<const float4*>(sv + hh * cols + cg * 4);
      const float4 wv = make_float4(w * v.x, w * v.y, w * v.z, w * v.w);
      float* dst = sp + hh * hs;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = bt * U * n_rg + rg + u * n_rg;
        if (r >= dk) break;
        const float kr = k[r], qr = q[r];
        s[u].x = d * s[u].x + kr * wv.x; s[u].y = d * s[u].y + kr * wv.y;
        s[u].z = d * s[u].z + kr * wv.z; s[u].w = d * s[u].w + kr * wv.w;
        *reinterpret_cast<float4*>(dst + (long long)r * a.dv) = s[u];
        o[0] += qr * s[u].x; o[1] += qr * s[u].y; o[2] += qr * s[u].z; o[3] += qr * s[u].w;
      }
    }
    if (bt == batches - 1) {                                  // the head's output: sums over the row groups
      float* rd = red + (hh & 1) * n_rg * cols;
      if (rg < n_rg) *reinterpret_cast<float4*>(rd + rg * cols + cg * 4) = make_float4(o[0], o[1], o[2], o[3]);
      o[0] = o[1] = o[2] = o[3] = 0.f;
      __syncthreads();
      for (int c = tid; c < my_cols; c += 256) {
        float acc = 0.f;
        for (int i = 0; i < n_rg; ++i) acc += rd[i * cols + c];
        out[hh * a.dv + c] = from_f<T>(acc * s_scale[hh] + s_skip[hh] * sv[hh * cols + c]);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) s[u] = nx[u];
  }
}

template <typename T, int KIND>
cudaError_t launch_step(const typename StepArgs<KIND>::type& p, int taps, int sm_count, cudaStream_t s) {
  const RecurrenceArgs& a = p.r;
  if (a.n_seq == 0) return cudaSuccess;
  // value columns per CTA: the whole head, or a part of it while that leaves SMs without work; then heads per CTA
  int cols = (a.dv + 31) / 32 * 32;
  while (cols > 32 && (long long)a.n_seq * a.heads * ((a.dv + cols - 1) / cols) < 2ll * sm_count) cols = (cols / 2 + 31) / 32 * 32;
  const long long ctas = (long long)a.n_seq * a.heads * ((a.dv + cols - 1) / cols);
  const int whole = KIND == kSsd ? a.kv_rep : a.heads, n_rg = 256 / (cols / 4);
  auto smem = [&](int hb) { return ((size_t)(KIND == kSsd ? 2 : 2 * hb) * ((a.dk + 3) & ~3) + (size_t)hb * cols + 2ull * n_rg * cols) * sizeof(float); };
  int hb = 1;
  while (hb < kMaxBlockHeads && whole % (2 * hb) == 0 && ctas / (2 * hb) >= 4ll * sm_count && smem(2 * hb) <= 40 * 1024) hb *= 2;
  const dim3 grid((unsigned)a.n_seq, (unsigned)(a.heads / hb), (unsigned)((a.dv + cols - 1) / cols));
  auto run = [&](auto kern) { kern<<<grid, 256, smem(hb), s>>>(p, cols, hb); };
  if (KIND == kSsd && taps == 4) run(recurrence_step_kernel<T, KIND, 4>);
  else if (KIND == kSsd && taps == 3) run(recurrence_step_kernel<T, KIND, 3>);
  else if (KIND == kSsd && taps == 2) run(recurrence_step_kernel<T, KIND, 2>);
  else run(recurrence_step_kernel<T, KIND, 0>);
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
cudaError_t launch_max_gate_step(const MaxGateStepArgs& a, int sm_count, cudaStream_t s) { return launch_step<T, kMaxGate>(a, 0, sm_count, s); }
template <typename T>
cudaError_t launch_ssd_step(const SsdStepArgs& a, int sm_count, cudaStream_t s) { return launch_step<T, kSsd>(a, a.taps, sm_count, s); }

#define FA_RECURRENCE(T)                                                           \
  template cudaError_t launch_recurrence_scan<T>(const RecurrenceArgs&, cudaStream_t); \
  template cudaError_t launch_max_gate_step<T>(const MaxGateStepArgs&, int, cudaStream_t); \
  template cudaError_t launch_ssd_step<T>(const SsdStepArgs&, int, cudaStream_t);
FA_RECURRENCE(bf16)
FA_RECURRENCE(float)

}  // namespace mixers
}  // namespace fa
