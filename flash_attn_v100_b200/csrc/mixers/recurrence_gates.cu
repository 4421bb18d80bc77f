// What the gated recurrences need per token before a prompt's state can be advanced, sm_100a: log decays and weights from the gate
// logits, and the short convolution.
#include "../hybrid/hybrid_common.cuh"
#include "recurrence.cuh"

namespace fa {
namespace mixers {

using hybrid::bf16;
using hybrid::from_f;
using hybrid::load_n;
using hybrid::silu_t;
using hybrid::store_n;
using hybrid::to_f;

namespace {

constexpr int kThreads = 256;

// ---- running maximum ----------------------------------------------------------------------------------------
// The map m -> max(m + F, M) of a run of tokens; runs compose.
struct MaxMap {
  float F, M;
};
__device__ __forceinline__ MaxMap then(const MaxMap& x, const MaxMap& y) { return {x.F + y.F, fmaxf(x.M + y.F, y.M)}; }

constexpr int kPer = 4;      // consecutive tokens per thread

// CTA = (sequence, head).  Tiles of 1024 tokens: a scan of the maps of the threads' tokens gives every thread the maximum before its
// first token.
template <typename T>
__global__ void __launch_bounds__(kThreads) max_gates_kernel(const MaxGateArgs a) {
  __shared__ MaxMap warp_map[kThreads / 32];
  const int seq = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  long long t0 = seq, t1 = seq + 1;
  if (a.cu != nullptr) {
    t0 = a.cu[seq];
    t1 = a.cu[seq + 1];
  }
  if (t0 < 0) t0 = 0;
  if (t1 > a.total) t1 = a.total;
  if (t1 <= t0) return;
  const int slot = a.slots[seq], start = a.starts[seq];
  const bool ok = slot >= 0 && slot < a.n_slots;
  if (!ok && tid == 0) atomicOr(a.status, 2);
  const bool fresh = start == 0 || !ok;
  const long long old_half = ((long long)slot * 2 + ((start - 1) & 1)) * a.heads + head;
  float m = fresh ? 0.f : a.m[old_half];           // before the tile's first token
  if (a.n0 != nullptr)
    for (int i = tid; i < a.dk; i += kThreads)
      a.n0[((long long)seq * a.heads + head) * a.dk + i] = fresh ? 0.f : a.norm[old_half * a.dk + i];
  const T* z = static_cast<const T*>(a.z);
  const float bi = to_f(static_cast<const T*>(a.bias_i)[head]), bf = to_f(static_cast<const T*>(a.bias_f)[head]);
  float zi[kPer], zf[kPer];
  auto fetch = [&](long long tile) {
#pragma unroll
    for (int u = 0; u < kPer; ++u) {
      const long long t = tile + tid * kPer + u;
      zi[u] = t < t1 ? to_f(z[t * a.stride + a.off_i + head]) : 0.f;
      zf[u] = t < t1 ? to_f(z[t * a.stride + a.off_f + head]) : 0.f;
    }
  };
  fetch(t0);
  for (long long tile = t0; tile < t1; tile += kThreads * kPer) {
    float gi[kPer], gf[kPer];
    MaxMap mine{0.f, -INFINITY};
#pragma unroll
    for (int u = 0; u < kPer; ++u) {
      gi[u] = a.cap * tanhf((zi[u] + bi) / a.cap);
      const float x = a.cap * tanhf((zf[u] + bf) / a.cap);
      gf[u] = x < 0.f ? x - log1pf(expf(x)) : -log1pf(expf(-x));
      if (tile + tid * kPer + u < t1) mine = then(mine, {gf[u], gi[u]});
    }
    if (tile + kThreads * kPer < t1) fetch(tile + kThreads * kPer);
    MaxMap scan = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      MaxMap prev{__shfl_up_sync(0xffffffffu, scan.F, o), __shfl_up_sync(0xffffffffu, scan.M, o)};
      if (lane >= o) scan = then(prev, scan);
    }
    if (lane == 31) warp_map[warp] = scan;
    MaxMap before{__shfl_up_sync(0xffffffffu, scan.F, 1), __shfl_up_sync(0xffffffffu, scan.M, 1)};
    __syncthreads();
    float mw = m, m_tile = m;
#pragma unroll
    for (int i = 0; i < kThreads / 32; ++i) {
      if (i == warp) mw = m_tile;
      m_tile = fmaxf(m_tile + warp_map[i].F, warp_map[i].M);
    }
    __syncthreads();
    float mt = lane == 0 ? mw : fmaxf(mw + before.F, before.M);
#pragma unroll
    for (int u = 0; u < kPer; ++u) {
      const long long t = tile + tid * kPer + u;
      if (t >= t1) break;
      const float mn = fmaxf(gf[u] + mt, gi[u]);
      const long long at = (long long)head * a.total + t;
      a.la[at] = gf[u] + mt - mn;
      a.b[at] = expf(gi[u] - mn);
      a.floor[at] = expf(-mn);
      if (t == t1 - 1 && ok) a.m[((long long)slot * 2 + ((start + (int)(t1 - t0) - 1) & 1)) * a.heads + head] = mn;
      mt = mn;
    }
    m = m_tile;
  }
}

// ---- step sizes -----------------------------------------------------------------------------------------------
// 32 tokens x 32 heads per CTA, turned in shared memory: the logits have the heads inside, the results the tokens.
template <typename T>
__global__ void __launch_bounds__(kThreads) step_gates_kernel(const StepGateArgs a) {
  __shared__ float tile[32][33];
  const long long t0 = (long long)blockIdx.x * 32;
  const int h0 = blockIdx.y * 32, x = threadIdx.x & 31, y = threadIdx.x >> 5;
  const T* z = static_cast<const T*>(a.z);
  for (int i = y; i < 32; i += kThreads / 32)
    if (t0 + i < a.total && h0 + x < a.heads) tile[i][x] = to_f(z[(t0 + i) * a.stride + a.off + h0 + x]);
  __syncthreads();
  for (int i = y; i < 32; i += kThreads / 32) {
    const int h = h0 + i;
    if (h >= a.heads || t0 + x >= a.total) continue;
    const float v = tile[x][i] + a.bias[h];
    const float dt = v > 0.f ? v + log1pf(expf(-v)) : log1pf(expf(v));
    const long long at = (long long)h * a.total + t0 + x;
    a.la[at] = -expf(a.a_log[h]) * dt;
    a.b[at] = dt;
  }
}

// ---- convolution ------------------------------------------------------------------------------------------------
constexpr int kRun = 16;     // consecutive tokens per thread

// A thread carries VEC channels through kRun tokens with the inputs of the last TAPS - 1 positions in registers (TAPS 0: any number of
// taps, every input is read again).
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(kThreads) conv_silu_kernel(const ConvArgs a) {
  const int nv = a.channels / VEC;
  const long long id = (long long)blockIdx.x * kThreads + threadIdx.x;
  const long long run = id / nv;
  const int c = (int)(id - run * nv) * VEC;
  const long long ta = run * kRun;
  if (ta >= a.total) return;
  const long long tb = ta + kRun < a.total ? ta + kRun : a.total;
  const T *z = static_cast<const T*>(a.z) + a.off + c, *wt = static_cast<const T*>(a.w) + c;
  const int taps = TAPS > 0 ? TAPS : a.taps;
  float bias[VEC];
  load_n<VEC>(static_cast<const T*>(a.bias) + c, bias);
  // input of the token `back` positions before token t of sequence seq (position pos, first token of the call seq0)
  auto input = [&](long long t, int back, int seq, int pos, long long seq0, float (&v)[VEC]) {
    if (t - back >= seq0) {
      load_n<VEC>(z + (t - back) * a.stride, v);
      return;
    }
    const int p = pos - back, slot = a.slots[seq];
    if (p >= 0 && slot >= 0 && slot < a.n_slots) {
      load_n<VEC>(static_cast<const T*>(a.ring) + ((long long)slot * taps + p % taps) * a.channels + c, v);
    } else {
      if (p >= 0 && c == 0) atomicOr(a.status, 2);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
    }
  };
  auto emit = [&](long long t, float (&acc)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) acc[i] = silu_t<T>(acc[i]);
    store_n<VEC>(static_cast<T*>(a.out) + t * a.channels + c, acc);
  };
  if constexpr (TAPS > 0) {
    float win[TAPS][VEC], wk[TAPS][VEC];     // win[k]: the input k positions back
#pragma unroll
    for (int k = 0; k < TAPS; ++k) load_n<VEC>(wt + (long long)(TAPS - 1 - k) * a.channels, wk[k]);
    auto advance = [&](long long t, const float (&in)[VEC]) {
      float acc[VEC];
#pragma unroll
      for (int k = TAPS - 1; k > 0; --k)
#pragma unroll
        for (int i = 0; i < VEC; ++i) win[k][i] = win[k - 1][i];
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        win[0][i] = in[i];
        acc[i] = bias[i];
      }
#pragma unroll
      for (int k = 0; k < TAPS; ++k)
#pragma unroll
        for (int i = 0; i < VEC; ++i) acc[i] += wk[k][i] * win[k][i];
      emit(t, acc);
    };
    int seq = -1;
    for (long long t = ta; t < tb;) {
      const int s = a.tok_seq[t], pos = a.positions[t];
      if (s < 0 || s >= a.n_seq) {
        if (c == 0) atomicOr(a.status, 2);
        seq = -1;
        ++t;
        continue;
      }
      if (s != seq) {                        // win[k] will be k + 1 positions back
        const long long seq0 = a.cu != nullptr ? a.cu[s] : t;
#pragma unroll
        for (int k = 1; k < TAPS; ++k) input(t, k, s, pos, seq0, win[k - 1]);
        seq = s;
      }
      constexpr int B = 4;                   // tokens whose inputs are fetched together
      if (t + B <= tb && a.tok_seq[t + B - 1] == s) {
        float in[B][VEC];
#pragma unroll
        for (int j = 0; j < B; ++j) load_n<VEC>(z + (t + j) * a.stride, in[j]);
#pragma unroll
        for (int j = 0; j < B; ++j) advance(t + j, in[j]);
        t += B;
      } else {
        float in[VEC];
        load_n<VEC>(z + t * a.stride, in);
        advance(t, in);
        ++t;
      }
    }
  } else {
    for (long long t = ta; t < tb; ++t) {
      const int s = a.tok_seq[t], pos = a.positions[t];
      if (s < 0 || s >= a.n_seq) {
        if (c == 0) atomicOr(a.status, 2);
        continue;
      }
      const long long seq0 = a.cu != nullptr ? a.cu[s] : t;
      float acc[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) acc[i] = bias[i];
      for (int k = 0; k < a.taps; ++k) {
        float w[VEC], in[VEC];
        load_n<VEC>(wt + (long long)(a.taps - 1 - k) * a.channels, w);
        input(t, k, s, pos, seq0, in);
#pragma unroll
        for (int i = 0; i < VEC; ++i) acc[i] += w[i] * in[i];
      }
      emit(t, acc);
    }
  }
}

// The inputs of a call's last `taps` positions go to the slot's ring, once the convolution has read what was there.
template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads) conv_keep_kernel(const ConvArgs a) {
  const int seq = blockIdx.x, back = blockIdx.y;
  long long t0 = seq, t1 = seq + 1;
  if (a.cu != nullptr) {
    t0 = a.cu[seq];
    t1 = a.cu[seq + 1];
  }
  if (t0 < 0) t0 = 0;
  if (t1 > a.total) t1 = a.total;
  const long long t = t1 - 1 - back;
  const int slot = a.slots[seq];
  if (t < t0 || slot < 0 || slot >= a.n_slots) return;
  const int pos = a.positions[t];
  if (pos < 0) return;
  const T* z = static_cast<const T*>(a.z) + t * a.stride + a.off;
  T* ring = static_cast<T*>(a.ring) + ((long long)slot * a.taps + pos % a.taps) * a.channels;
  for (int c = threadIdx.x * VEC; c < a.channels; c += kThreads * VEC) {
    float v[VEC];
    load_n<VEC>(z + c, v);
    store_n<VEC>(ring + c, v);
  }
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T, int VEC>
cudaError_t launch_conv_t(const ConvArgs& a, cudaStream_t s) {
  const long long threads = (a.total + kRun - 1) / kRun * (a.channels / VEC);
  const unsigned grid = (unsigned)((threads + kThreads - 1) / kThreads);
  switch (a.taps) {
    case 2: conv_silu_kernel<T, VEC, 2><<<grid, kThreads, 0, s>>>(a); break;
    case 3: conv_silu_kernel<T, VEC, 3><<<grid, kThreads, 0, s>>>(a); break;
    case 4: conv_silu_kernel<T, VEC, 4><<<grid, kThreads, 0, s>>>(a); break;
    default: conv_silu_kernel<T, VEC, 0><<<grid, kThreads, 0, s>>>(a); break;
  }
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return e;
  conv_keep_kernel<T, VEC><<<dim3((unsigned)a.n_seq, (unsigned)a.taps), kThreads, 0, s>>>(a);
  return cudaGetLastError();
}

}  // namespace

template <typename T>
cudaError_t launch_max_gates(const MaxGateArgs& a, cudaStream_t s) {
  if (a.n_seq == 0) return cudaSuccess;
  max_gates_kernel<T><<<dim3((unsigned)a.n_seq, (unsigned)a.heads), kThreads, 0, s>>>(a);
  return cudaGetLastError();
}

template <typename T>
cudaError_t launch_step_gates(const StepGateArgs& a, cudaStream_t s) {
  if (a.total == 0) return cudaSuccess;
  step_gates_kernel<T><<<dim3((unsigned)((a.total + 31) / 32), (unsigned)((a.heads + 31) / 32)), kThreads, 0, s>>>(a);
  return cudaGetLastError();
}

template <typename T>
cudaError_t launch_conv_silu(const ConvArgs& a, cudaStream_t s) {
  if (a.total == 0 || a.n_seq == 0) return cudaSuccess;
  const bool vec = a.channels % 8 == 0 && a.stride % 8 == 0 && a.off % 8 == 0 && aligned16(a.z) && aligned16(a.w) && aligned16(a.bias) &&
                   aligned16(a.ring) && aligned16(a.out);
  return vec ? launch_conv_t<T, 8>(a, s) : launch_conv_t<T, 1>(a, s);
}

#define FA_GATES(T)                                                    \
  template cudaError_t launch_max_gates<T>(const MaxGateArgs&, cudaStream_t);   \
  template cudaError_t launch_step_gates<T>(const StepGateArgs&, cudaStream_t); \
  template cudaError_t launch_conv_silu<T>(const ConvArgs&, cudaStream_t);
FA_GATES(bf16)
FA_GATES(float)

}  // namespace mixers
}  // namespace fa
