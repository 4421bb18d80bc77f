// Preparation of the latent attention's cached rows, and rotation of query heads, sm_100a.
#include "hybrid_common.cuh"
#include "latent_prep.cuh"

namespace fa {
namespace hybrid {
namespace {

constexpr int kThreads = 256;

// One CTA per row: norms of the two latents, rotation of the shared key part, append of (latent, rotated part) to the
// row's place in the paged cache.  NQ / NK: vectors per thread that hold the query / key-value latent between the sum of squares
// and the scaling (0: any size, the row is read twice).
template <typename T, int VEC, int NQ, int NK>
__global__ void __launch_bounds__(kThreads) latent_prep_kernel(const LatentPrepArgs a) {
  __shared__ float red[2][kThreads / 32];
  const long long row = blockIdx.x;
  const int tid = threadIdx.x;
  const T* in = static_cast<const T*>(a.down) + row * a.down_stride;
  const T *zq = in + a.off_q, *zk = in + a.off_kv, *zr = in + a.off_r;
  const int nq = a.q_rank / VEC, nk = a.kv_rank / VEC, half = a.rot_dim / 2;
  float kq[NQ > 0 ? NQ : 1][VEC], kk[NK > 0 ? NK : 1][VEC];
  float sq = 0.f, sk = 0.f;
  auto add = [](float& s, const float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) s += v[i] * v[i];
  };
  if constexpr (NQ > 0) {
#pragma unroll
    for (int n = 0; n < NQ; ++n)
      if (tid + n * kThreads < nq) load_n<VEC>(zq + (tid + n * kThreads) * VEC, kq[n]);
#pragma unroll
    for (int n = 0; n < NK; ++n)
      if (tid + n * kThreads < nk) load_n<VEC>(zk + (tid + n * kThreads) * VEC, kk[n]);
  }
  T* pool_row = nullptr;
  {
    const int seq = a.tok_seq[row], pos = a.positions[row];
    const int blk = pos >> 4;
    int page = -1;
    if (seq >= 0 && seq < a.n_seq && pos >= 0 && blk < a.max_blocks) page = a.block_table[(long long)seq * a.max_blocks + blk];
    if (page >= 0 && page < a.n_blocks) {
      pool_row = static_cast<T*>(a.pool) + ((long long)page * 16 + (pos & 15)) * a.pool_stride;
    } else if (tid == 0) {
      atomicOr(a.status, 2);
    }
  }
  T* r_out = a.r_out ? static_cast<T*>(a.r_out) + row * a.rot_dim : nullptr;
  for (int i = tid; i < half; i += kThreads) {
    const float cs = a.cos_t[row * half + i], sn = a.sin_t[row * half + i];
    const float u = to_f(zr[i]), v = to_f(zr[i + half]);
    const T ru = from_f<T>(u * cs - v * sn), rv = from_f<T>(v * cs + u * sn);
    if (pool_row) { pool_row[a.kv_rank + i] = ru; pool_row[a.kv_rank + half + i] = rv; }
    if (r_out) { r_out[i] = ru; r_out[half + i] = rv; }
  }
  if constexpr (NQ > 0) {
#pragma unroll
    for (int n = 0; n < NQ; ++n)
      if (tid + n * kThreads < nq) add(sq, kq[n]);
#pragma unroll
    for (int n = 0; n < NK; ++n)
      if (tid + n * kThreads < nk) add(sk, kk[n]);
  } else {
    for (int c = tid; c < nq; c += kThreads) { load_n<VEC>(zq + c * VEC, kq[0]); add(sq, kq[0]); }
    for (int c = tid; c < nk; c += kThreads) { load_n<VEC>(zk + c * VEC, kk[0]); add(sk, kk[0]); }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) { sq += red[0][i]; sk += red[1][i]; }
  const float qinv = 1.f / sqrtf(sq / (float)a.q_rank + a.eps), kinv = 1.f / sqrtf(sk / (float)a.kv_rank + a.eps);
  T* cq = static_cast<T*>(a.cq) + row * a.q_rank;
  T* c_out = a.c_out ? static_cast<T*>(a.c_out) + row * a.kv_rank : nullptr;
  const T *wq = static_cast<const T*>(a.wq), *wkv = static_cast<const T*>(a.wkv);
  auto scale = [](float (&v)[VEC], float inv, const T* w) {
    float wv[VEC];
    load_n<VEC>(w, wv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = v[i] * inv * wv[i];
  };
  auto emit_q = [&](int c, float (&v)[VEC]) {
    scale(v, qinv, wq + c * VEC);
    store_n<VEC>(cq + c * VEC, v);
  };
  auto emit_k = [&](int c, float (&v)[VEC]) {
    scale(v, kinv, wkv + c * VEC);
    if (pool_row) store_n<VEC>(pool_row + c * VEC, v);
    if (c_out) store_n<VEC>(c_out + c * VEC, v);
  };
  if constexpr (NQ > 0) {
#pragma unroll
    for (int n = 0; n < NQ; ++n)
      if (tid + n * kThreads < nq) emit_q(tid + n * kThreads, kq[n]);
#pragma unroll
    for (int n = 0; n < NK; ++n)
      if (tid + n * kThreads < nk) emit_k(tid + n * kThreads, kk[n]);
  } else {
    for (int c = tid; c < nq; c += kThreads) { load_n<VEC>(zq + c * VEC, kq[0]); emit_q(c, kq[0]); }
    for (int c = tid; c < nk; c += kThreads) { load_n<VEC>(zk + c * VEC, kk[0]); emit_k(c, kk[0]); }
  }
}

// In-place rotation of columns [off, off + rot_dim) of every head; q [rows, heads * head_stride].
template <typename T>
__global__ void __launch_bounds__(kThreads) rotate_heads_kernel(T* q, const float* cos_t, const float* sin_t, long long rows,
                                                               int heads, int head_stride, int off, int rot_dim) {
  const int half = rot_dim / 2;
  const long long total = rows * heads * half;
  for (long long i = (long long)blockIdx.x * kThreads + threadIdx.x; i < total; i += (long long)gridDim.x * kThreads) {
    const long long rh = i / half;
    const int c = (int)(i - rh * half);
    const long long row = rh / heads;
    T* p = q + rh * head_stride + off;
    const float cs = cos_t[row * half + c], sn = sin_t[row * half + c];
    const float u = to_f(p[c]), v = to_f(p[c + half]);
    p[c] = from_f<T>(u * cs - v * sn);
    p[c + half] = from_f<T>(v * cs + u * sn);
  }
}

unsigned grid_1d(long long threads) {
  long long blocks = (threads + kThreads - 1) / kThreads;
  if (blocks > 148 * 32) blocks = 148 * 32;
  return (unsigned)(blocks < 1 ? 1 : blocks);
}
bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

template <typename T>
cudaError_t launch_latent_prep(const LatentPrepArgs& a, cudaStream_t s) {
  if (a.rows == 0) return cudaSuccess;
  const unsigned g = (unsigned)a.rows;
  const bool vec = a.q_rank % 8 == 0 && a.kv_rank % 8 == 0 && a.off_q % 8 == 0 && a.off_kv % 8 == 0 && a.down_stride % 8 == 0 &&
                   a.pool_stride % 8 == 0 && aligned16(a.down) && aligned16(a.wq) && aligned16(a.wkv) && aligned16(a.cq) &&
                   aligned16(a.c_out) && aligned16(a.pool);
  if (vec && a.q_rank <= 8 * kThreads && a.kv_rank <= 8 * kThreads) latent_prep_kernel<T, 8, 1, 1><<<g, kThreads, 0, s>>>(a);
  else if (vec) latent_prep_kernel<T, 8, 0, 0><<<g, kThreads, 0, s>>>(a);
  else latent_prep_kernel<T, 1, 0, 0><<<g, kThreads, 0, s>>>(a);
  return cudaGetLastError();
}

template <typename T>
cudaError_t launch_rotate_heads(void* q, const float* cos_t, const float* sin_t, long long rows, int heads, int head_stride, int off,
                                int rot_dim, cudaStream_t s) {
  if (rows == 0 || rot_dim == 0) return cudaSuccess;
  rotate_heads_kernel<T><<<grid_1d(rows * heads * (rot_dim / 2)), kThreads, 0, s>>>(static_cast<T*>(q), cos_t, sin_t, rows, heads,
                                                                                  head_stride, off, rot_dim);
  return cudaGetLastError();
}

#define FA_LATENT_PREP(T)                                                          \
  template cudaError_t launch_latent_prep<T>(const LatentPrepArgs&, cudaStream_t); \
  template cudaError_t launch_rotate_heads<T>(void*, const float*, const float*, long long, int, int, int, int, cudaStream_t);
FA_LATENT_PREP(bf16)
FA_LATENT_PREP(float)

}  // namespace hybrid
}  // namespace fa
