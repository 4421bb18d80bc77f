// Grouped-query attention on paged keys and values, sm_100a: preparation of queries, keys and values, the general kernel (any
// size, bfloat16 or float), and the gather of cached rows.
#include <math_constants.h>

#include "../hybrid/hybrid_common.cuh"
#include "kv_attention.cuh"

namespace fa {
namespace mixers {

using hybrid::bf16;
using hybrid::from_f;
using hybrid::load_n;
using hybrid::sigmoid_f;
using hybrid::store_n;
using hybrid::to_f;
using hybrid::warp_max;
using hybrid::warp_sum;

namespace {

constexpr int kThreads = 256;

// One CTA per row: both norms, value mixing, append to the row's place in the pages.  NQ: vectors per thread that hold the queries
// between the sum of squares and the scaling (0: any size, the row is read twice); keys: one vector, or any number with NQ = 0.
template <typename T, int VEC, int NQ>
__global__ void __launch_bounds__(kThreads) kv_prep_kernel(const KvPrepArgs a) {
  __shared__ float red[2][kThreads / 32];
  const long long row = blockIdx.x;
  const int tid = threadIdx.x;
  const T* in = static_cast<const T*>(a.z) + row * a.stride;
  const T *zq = in + a.off_q, *zk = in + a.off_k, *zv = in + a.off_v;
  const int cq = a.heads * a.dim, ck = a.kv_heads * a.dim, cv = a.kv_heads * a.vdim;
  const int nq = cq / VEC, nk = ck / VEC, nv = cv / VEC;
  long long page = -1;
  int slot = 0;
  {
    const int seq = a.pg.tok_seq[row], pos = a.pg.positions[row];
    if (seq >= 0 && seq < a.pg.n_seq && pos >= 0 && (pos >> 4) < a.pg.max_blocks) page = a.pg.block_table[(long long)seq * a.pg.max_blocks + (pos >> 4)];
    slot = pos & 15;
    if (page < 0 || page >= a.pg.n_blocks) {
      page = -1;
      if (tid == 0) atomicOr(a.status, 2);
    }
  }
  float kq[NQ > 0 ? NQ : 1][VEC], kk[VEC];
  float sq = 0.f, sk = 0.f;
  auto add = [](float& s, const float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) s += v[i] * v[i];
  };
  if constexpr (NQ > 0) {
#pragma unroll
    for (int n = 0; n < NQ; ++n)
      if (tid + n * kThreads < nq) { load_n<VEC>(zq + (tid + n * kThreads) * VEC, kq[n]); add(sq, kq[n]); }
    if (tid < nk) { load_n<VEC>(zk + tid * VEC, kk); add(sk, kk); }
  } else {
    for (int c = tid; c < nq; c += kThreads) { load_n<VEC>(zq + c * VEC, kq[0]); add(sq, kq[0]); }
    for (int c = tid; c < nk; c += kThreads) { load_n<VEC>(zk + c * VEC, kk); add(sk, kk); }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) { sq += red[0][i]; sk += red[1][i]; }
  const float iq = 1.f / sqrtf(sq / (float)cq + a.eps), ik = 1.f / sqrtf(sk / (float)ck + a.eps);
  T* q = static_cast<T*>(a.q) + row * cq;
  T* k = a.k != nullptr ? static_cast<T*>(a.k) + row * ck : nullptr;
  T* v = a.v != nullptr ? static_cast<T*>(a.v) + row * cv : nullptr;
  auto emit_q = [&](int c, float (&x)[VEC]) {
    float w[VEC];
    load_n<VEC>(static_cast<const T*>(a.wq) + c * VEC, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[i] = x[i] * iq * w[i];
    store_n<VEC>(q + c * VEC, x);
  };
  auto emit_k = [&](int c, float (&x)[VEC]) {
    float w[VEC];
    load_n<VEC>(static_cast<const T*>(a.wk) + c * VEC, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[i] = x[i] * ik * w[i];
    if (k != nullptr) store_n<VEC>(k + c * VEC, x);
    const int h = c * VEC / a.dim, d = c * VEC - h * a.dim;
    if (page >= 0) store_n<VEC>(static_cast<T*>(a.k_pool) + ((page * a.kv_heads + h) * 16 + slot) * a.dim + d, x);
  };
  if constexpr (NQ > 0) {
#pragma unroll
    for (int n = 0; n < NQ; ++n)
      if (tid + n * kThreads < nq) emit_q(tid + n * kThreads, kq[n]);
    if (tid < nk) emit_k(tid, kk);
  } else {
    for (int c = tid; c < nq; c += kThreads) { load_n<VEC>(zq + c * VEC, kq[0]); emit_q(c, kq[0]); }
    for (int c = tid; c < nk; c += kThreads) { load_n<VEC>(zk + c * VEC, kk); emit_k(c, kk); }
  }
  const T* first = a.v_first != nullptr ? static_cast<const T*>(a.v_first) + row * a.first_stride : nullptr;
  for (int c = tid; c < nv; c += kThreads) {
    float x[VEC];
    load_n<VEC>(zv + c * VEC, x);
    if (first != nullptr) {
      float y[VEC];
      load_n<VEC>(first + c * VEC, y);
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[i] = (1.f - a.lambda) * x[i] + a.lambda * y[i];
    }
    if (v != nullptr) store_n<VEC>(v + c * VEC, x);
    const int h = c * VEC / a.vdim, d = c * VEC - h * a.vdim;
    if (page >= 0) store_n<VEC>(static_cast<T*>(a.v_pool) + ((page * a.kv_heads + h) * 16 + slot) * a.vdim + d, x);
  }
}

constexpr int kTile = 128;     // keys per step = threads per CTA of the general kernel

template <typename T>
__global__ void __launch_bounds__(kTile) kv_attention_kernel(const KvAttentionArgs a) {
  extern __shared__ float sm[];
  float* q = sm;                 // [dim]
  float* acc = q + a.dim;        // [vdim]
  float* p = acc + a.vdim;       // [kTile]
  float* red = p + kTile;        // [8]
  long long* rows = reinterpret_cast<long long*>(red + 8 + ((a.dim + a.vdim) & 1));   // [kTile] row of the pools, or -1
  const long long row = blockIdx.x;
  const int head = blockIdx.y, tid = threadIdx.x, kvh = head / (a.heads / a.kv_heads);
  const T* qr = static_cast<const T*>(a.q) + (row * a.heads + head) * a.dim;
  for (int c = tid; c < a.dim; c += kTile) q[c] = to_f(qr[c]) * a.scale;
  for (int c = tid; c < a.vdim; c += kTile) acc[c] = 0.f;
  const int seq = a.pg.tok_seq[row], pos = a.pg.positions[row];
  int n = pos + 1;
  bool bad = seq < 0 || seq >= a.pg.n_seq || n <= 0 || (n + 15) / 16 > a.pg.max_blocks;
  if (bad) n = 0;
  const int first = a.chunk > 0 && n > 0 ? pos - pos % a.chunk : 0;
  const float slope = a.slopes != nullptr ? a.slopes[head] : 0.f;
  float m = -CUDART_INF_F, l = 0.f;
  for (int k0 = first; k0 < n; k0 += kTile) {
    const int key = k0 + tid;
    long long kr = -1;
    if (key < n) {
      const int page = a.pg.block_table[(long long)seq * a.pg.max_blocks + (key >> 4)];
      if (page >= 0 && page < a.pg.n_blocks) kr = ((long long)page * a.kv_heads + kvh) * 16 + (key & 15);
      else bad = true;
    }
    __syncthreads();             // q is complete; the previous step's p and rows are no longer read
    float s = -CUDART_INF_F;
    if (kr >= 0) {
      const T* kp = static_cast<const T*>(a.k_pool) + kr * a.dim;
      s = 0.f;
      for (int c = 0; c < a.dim; ++c) s += q[c] * to_f(kp[c]);
      s -= slope * (float)(pos - key);
    }
    rows[tid] = kr;
    float mx = warp_max(s);
    if ((tid & 31) == 0) red[tid >> 5] = mx;
    __syncthreads();
    mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    const float m_new = fmaxf(m, mx);
    const float w = kr >= 0 ? expf(s - m_new) : 0.f;
    p[tid] = w;
    const float ws = warp_sum(w);
    if ((tid & 31) == 0) red[4 + (tid >> 5)] = ws;
    const float f = m == -CUDART_INF_F ? 0.f : expf(m - m_new);
    __syncthreads();
    l = l * f + red[4] + red[5] + red[6] + red[7];
    m = m_new;
    const int cnt = n - k0 < kTile ? n - k0 : kTile;
    for (int c = tid; c < a.vdim; c += kTile) {
      float o = acc[c] * f;
      for (int j = 0; j < cnt; ++j)
        if (rows[j] >= 0) o += p[j] * to_f(static_cast<const T*>(a.v_pool)[rows[j] * a.vdim + c]);
      acc[c] = o;
    }
  }
  __syncthreads();
  if (bad) atomicOr(a.status, 2);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  const T* g = a.gate != nullptr ? static_cast<const T*>(a.gate) + row * a.gate_stride + head * a.vdim : nullptr;
  T* out = static_cast<T*>(a.out) + row * a.out_stride + head * a.vdim;
  for (int c = tid; c < a.vdim; c += kTile) out[c] = from_f<T>(acc[c] * inv * (g != nullptr ? sigmoid_f(to_f(g[c])) : 1.f));
}

// One warp per row: a cached position's keys and values of all heads to contiguous rows.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) kv_gather_kernel(const KvGatherArgs a) {
  const long long row = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (row >= a.total_kv) return;
  int lo = 0, hi = a.pieces - 1;                // last piece that starts at or before the row
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (a.cu_kv[mid] <= row) lo = mid; else hi = mid - 1;
  }
  const int seq = a.piece_seq[lo], pos = a.piece_key0[lo] + (int)(row - a.cu_kv[lo]);
  int page = -1;
  if (seq >= 0 && seq < a.n_seq && pos >= 0 && (pos >> 4) < a.max_blocks) page = a.block_table[(long long)seq * a.max_blocks + (pos >> 4)];
  const bool ok = page >= 0 && page < a.n_blocks;
  if (!ok && lane == 0) atomicOr(a.status, 2);
  auto copy = [&](const void* pool, void* dst, int dim) {
    const int n = a.kv_heads * dim;
    T* d = static_cast<T*>(dst) + row * n;
    for (int c = lane * VEC; c < n; c += 32 * VEC) {
      const int h = c / dim;
      float v[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
      if (ok) load_n<VEC>(static_cast<const T*>(pool) + (((long long)page * a.kv_heads + h) * 16 + (pos & 15)) * dim + c - h * dim, v);
      store_n<VEC>(d + c, v);
    }
  };
  copy(a.k_pool, a.k, a.dim);
  copy(a.v_pool, a.v, a.vdim);
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

template <typename T>
cudaError_t launch_kv_prep(const KvPrepArgs& a, cudaStream_t s) {
  if (a.rows == 0) return cudaSuccess;
  const unsigned g = (unsigned)a.rows;
  const int cq = a.heads * a.dim, ck = a.kv_heads * a.dim;
  const bool vec = a.dim % 8 == 0 && a.vdim % 8 == 0 && a.off_q % 8 == 0 && a.off_k % 8 == 0 && a.off_v % 8 == 0 && a.stride % 8 == 0 &&
                   aligned16(a.z) && aligned16(a.wq) && aligned16(a.wk) && aligned16(a.q) && aligned16(a.k) && aligned16(a.v) &&
                   aligned16(a.k_pool) && aligned16(a.v_pool) && (a.v_first == nullptr || (aligned16(a.v_first) && a.first_stride % 8 == 0));
  if (vec && cq <= 8 * kThreads && ck <= 8 * kThreads) kv_prep_kernel<T, 8, 1><<<g, kThreads, 0, s>>>(a);
  else if (vec && cq <= 16 * kThreads && ck <= 8 * kThreads) kv_prep_kernel<T, 8, 2><<<g, kThreads, 0, s>>>(a);
  else if (vec && cq <= 32 * kThreads && ck <= 8 * kThreads) kv_prep_kernel<T, 8, 4><<<g, kThreads, 0, s>>>(a);
  else if (vec) kv_prep_kernel<T, 8, 0><<<g, kThreads, 0, s>>>(a);
  else kv_prep_kernel<T, 1, 0><<<g, kThreads, 0, s>>>(a);
  return cudaGetLastError();
}

template <typename T>
cudaError_t launch_kv_attention(const KvAttentionArgs& a, cudaStream_t s) {
  if (a.rows == 0) return cudaSuccess;
  const size_t smem = ((size_t)a.dim + a.vdim + kTile + 8 + 1) * sizeof(float) + kTile * sizeof(long long);
  cudaError_t e = cudaFuncSetAttribute(kv_attention_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  kv_attention_kernel<T><<<dim3((unsigned)a.rows, (unsigned)a.heads), kTile, smem, s>>>(a);
  return cudaGetLastError();
}

template <typename T>
cudaError_t launch_kv_gather(const KvGatherArgs& a, cudaStream_t s) {
  if (a.total_kv == 0) return cudaSuccess;
  const unsigned g = (unsigned)((a.total_kv + 7) / 8);
  if (a.dim % 8 == 0 && a.vdim % 8 == 0 && aligned16(a.k_pool) && aligned16(a.v_pool) && aligned16(a.k) && aligned16(a.v))
    kv_gather_kernel<T, 8><<<g, 256, 0, s>>>(a);
  else
    kv_gather_kernel<T, 1><<<g, 256, 0, s>>>(a);
  return cudaGetLastError();
}

#define FA_KV(T)                                                          \
  template cudaError_t launch_kv_prep<T>(const KvPrepArgs&, cudaStream_t);           \
  template cudaError_t launch_kv_attention<T>(const KvAttentionArgs&, cudaStream_t); \
  template cudaError_t launch_kv_gather<T>(const KvGatherArgs&, cudaStream_t);
FA_KV(bf16)
FA_KV(float)

}  // namespace mixers
}  // namespace fa
