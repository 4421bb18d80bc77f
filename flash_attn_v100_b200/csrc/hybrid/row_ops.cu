// Row-wise operators of the hybrid decoder, sm_100a: residual update + RMS norm, gated output norm, clamped gated
// feed-forward activation, token side input, and the preparation of the latent attention's cached rows.
//
// The residual stream is fp32; activations are T (bfloat16 or float).  Every operator is one pass over its rows
// (HBM-bound); the vector width is chosen at launch from the sizes, so that any width runs.
#include "hybrid_common.cuh"
#include "row_ops.cuh"

namespace fa {
namespace hybrid {
namespace {

constexpr int kThreads = 256;

// KEEP: vectors per thread that stay in registers between the passes over a row (0: the row is read again).
// x (+)= [embedding] + [delta or rmsnorm(delta) * delta_w]; out = rmsnorm(x) * w (or x).  One CTA per row.
template <typename T, int VEC, int KEEP>
__global__ void __launch_bounds__(kThreads) residual_norm_kernel(const ResidualNormArgs a) {
  __shared__ float red[kThreads / 32];
  const long long row = blockIdx.x;
  float* x = a.x + row * a.cols;
  const T* d = a.delta ? static_cast<const T*>(a.delta) + row * a.cols : nullptr;
  const T* dw = static_cast<const T*>(a.delta_w);
  const T* e = nullptr;
  if (a.embed_mode != 0) {
    int64_t tok = a.tokens[row];
    tok = tok < 0 ? 0 : (tok >= a.vocab ? a.vocab - 1 : tok);
    e = static_cast<const T*>(a.embed) + tok * a.cols;
  }
  const int nv = a.cols / VEC;
  float keep[KEEP > 0 ? KEEP : 1][VEC];
  float dinv = 1.f;
  if (d != nullptr && dw != nullptr) {
    float ss = 0.f;
#pragma unroll 4
    for (int c = threadIdx.x; c < nv; c += kThreads) {
      float v[VEC];
      load_n<VEC>(d + c * VEC, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss += v[i] * v[i];
    }
    dinv = 1.f / sqrtf(block_sum(ss, red) / (float)a.cols + a.eps);
  }
  auto updated = [&](int c, float (&v)[VEC]) {
    if (a.embed_mode == 2) {
      load_n<VEC>(e + c * VEC, v);
    } else {
      load_n<VEC>(x + c * VEC, v);
    }
    if (d != nullptr) {
      float t[VEC];
      load_n<VEC>(d + c * VEC, t);
      if (dw != nullptr) {
        float wv[VEC];
        load_n<VEC>(dw + c * VEC, wv);
#pragma unroll
        for (int i = 0; i < VEC; ++i) t[i] = t[i] * dinv * wv[i];
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] += t[i];
    }
    if (a.embed_mode == 1) {
      float t[VEC];
      load_n<VEC>(e + c * VEC, t);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] += t[i];
    }
  };
  const bool changed = d != nullptr || e != nullptr;
  float ss = 0.f;
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int n = 0; n < KEEP; ++n) {
      const int c = threadIdx.x + n * kThreads;
      if (c < nv) {
        updated(c, keep[n]);
        if (changed) store_n<VEC>(x + c * VEC, keep[n]);
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss += keep[n][i] * keep[n][i];
      }
    }
  } else {
    for (int c = threadIdx.x; c < nv; c += kThreads) {
      updated(c, keep[0]);
      if (changed) store_n<VEC>(x + c * VEC, keep[0]);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss += keep[0][i] * keep[0][i];
    }
  }
  if (a.out == nullptr) return;
  T* out = static_cast<T*>(a.out) + row * a.cols;
  const T* w = static_cast<const T*>(a.w);
  float inv = 1.f;
  if (w != nullptr) inv = 1.f / sqrtf(block_sum(ss, red) / (float)a.cols + a.eps);
  auto emit = [&](int c, float (&v)[VEC]) {
    if (w != nullptr) {
      float wv[VEC];
      load_n<VEC>(w + c * VEC, wv);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = v[i] * inv * wv[i];
    }
    store_n<VEC>(out + c * VEC, v);
  };
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int n = 0; n < KEEP; ++n) {
      const int c = threadIdx.x + n * kThreads;
      if (c < nv) emit(c, keep[n]);
    }
  } else {
    for (int c = threadIdx.x; c < nv; c += kThreads) {
      load_n<VEC>(x + c * VEC, keep[0]);     // this thread's own stores
      emit(c, keep[0]);
    }
  }
}

// out = rmsnorm(o) * w * sigmoid(g), the norm taken over the whole row.  One CTA per row.
template <typename T, int VEC, int KEEP>
__global__ void __launch_bounds__(kThreads) gated_norm_kernel(const T* o, const T* g, long long g_stride, const T* w, T* out,
                                                             int cols, float eps) {
  __shared__ float red[kThreads / 32];
  const long long row = blockIdx.x;
  o += row * cols; g += row * g_stride; out += row * cols;
  const int nv = cols / VEC;
  float keep[KEEP > 0 ? KEEP : 1][VEC];
  float ss = 0.f;
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int n = 0; n < KEEP; ++n) {
      const int c = threadIdx.x + n * kThreads;
      if (c < nv) {
        load_n<VEC>(o + c * VEC, keep[n]);
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss += keep[n][i] * keep[n][i];
      }
    }
  } else {
    for (int c = threadIdx.x; c < nv; c += kThreads) {
      load_n<VEC>(o + c * VEC, keep[0]);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss += keep[0][i] * keep[0][i];
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)cols + eps);
  auto emit = [&](int c, float (&v)[VEC]) {
    float wv[VEC], gv[VEC];
    load_n<VEC>(w + c * VEC, wv);
    load_n<VEC>(g + c * VEC, gv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = v[i] * inv * wv[i] * sigmoid_f(gv[i]);
    store_n<VEC>(out + c * VEC, v);
  };
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int n = 0; n < KEEP; ++n) {
      const int c = threadIdx.x + n * kThreads;
      if (c < nv) emit(c, keep[n]);
    }
  } else {
    for (int c = threadIdx.x; c < nv; c += kThreads) {
      load_n<VEC>(o + c * VEC, keep[0]);
      emit(c, keep[0]);
    }
  }
}

// gu [rows, 2n] (gate, then linear branch): out = g sigmoid(alpha g) (u + shift), g = min(gate, limit),
// u = clamp(linear, -limit, limit).
template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads) clamped_glu_kernel(const T* gu, T* out, long long rows, int n, float limit,
                                                              float alpha, float shift) {
  const int nv = n / VEC;
  const long long total = rows * nv;
  for (long long i = (long long)blockIdx.x * kThreads + threadIdx.x; i < total; i += (long long)gridDim.x * kThreads) {
    const long long row = i / nv;
    const int c = (int)(i - row * nv) * VEC;
    float g[VEC], u[VEC];
    load_n<VEC>(gu + row * 2 * n + c, g);
    load_n<VEC>(gu + row * 2 * n + n + c, u);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const float gg = fminf(g[j], limit), uu = fminf(fmaxf(u[j], -limit), limit);
      g[j] = gg * sigmoid_f(alpha * gg) * (uu + shift);
    }
    store_n<VEC>(out + row * n + c, g);
  }
}

// out = gelu_tanh(z) * side[token, off : off + n]
template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads) side_gate_kernel(const T* z, const T* side, const int64_t* tokens, int vocab,
                                                            long long side_stride, int off, T* out, long long rows, int n) {
  const int nv = n / VEC;
  const long long total = rows * nv;
  for (long long i = (long long)blockIdx.x * kThreads + threadIdx.x; i < total; i += (long long)gridDim.x * kThreads) {
    const long long row = i / nv;
    const int c = (int)(i - row * nv) * VEC;
    int64_t tok = tokens[row];
    tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
    float a[VEC], e[VEC];
    load_n<VEC>(z + row * n + c, a);
    load_n<VEC>(side + tok * side_stride + off + c, e);
#pragma unroll
    for (int j = 0; j < VEC; ++j) a[j] = gelu_tanh_f(a[j]) * e[j];
    store_n<VEC>(out + row * n + c, a);
  }
}

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
cudaError_t launch_residual_norm(const ResidualNormArgs& a, cudaStream_t s) {
  if (a.rows == 0) return cudaSuccess;
  const unsigned g = (unsigned)a.rows;
  const bool vec = a.cols % 4 == 0 && aligned16(a.x) && aligned16(a.delta) && aligned16(a.delta_w) && aligned16(a.embed) &&
                   aligned16(a.w) && aligned16(a.out);
  if (vec && a.cols <= 4 * kThreads) residual_norm_kernel<T, 4, 1><<<g, kThreads, 0, s>>>(a);
  else if (vec && a.cols <= 16 * kThreads) residual_norm_kernel<T, 4, 4><<<g, kThreads, 0, s>>>(a);
  else if (vec && a.cols <= 32 * kThreads) residual_norm_kernel<T, 4, 8><<<g, kThreads, 0, s>>>(a);
  else if (vec) residual_norm_kernel<T, 4, 0><<<g, kThreads, 0, s>>>(a);
  else residual_norm_kernel<T, 1, 0><<<g, kThreads, 0, s>>>(a);
  return cudaGetLastError();
}

template <typename T>
cudaError_t launch_gated_norm(const void* o, const void* g, long long g_stride, const void* w, void* out, long long rows, int cols,
                              float eps, cudaStream_t s) {
  if (rows == 0) return cudaSuccess;
  const T *op = static_cast<const T*>(o), *gp = static_cast<const T*>(g), *wp = static_cast<const T*>(w);
  T* outp = static_cast<T*>(out);
  const bool vec = cols % 8 == 0 && g_stride % 8 == 0 && aligned16(o) && aligned16(g) && aligned16(w) && aligned16(out);
  const unsigned grid = (unsigned)rows;
  if (vec && cols <= 8 * kThreads) gated_norm_kernel<T, 8, 1><<<grid, kThreads, 0, s>>>(op, gp, g_stride, wp, outp, cols, eps);
  else if (vec && cols <= 16 * kThreads) gated_norm_kernel<T, 8, 2><<<grid, kThreads, 0, s>>>(op, gp, g_stride, wp, outp, cols, eps);
  else if (vec && cols <= 32 * kThreads) gated_norm_kernel<T, 8, 4><<<grid, kThreads, 0, s>>>(op, gp, g_stride, wp, outp, cols, eps);
  else if (vec) gated_norm_kernel<T, 8, 0><<<grid, kThreads, 0, s>>>(op, gp, g_stride, wp, outp, cols, eps);
  else gated_norm_kernel<T, 1, 0><<<grid, kThreads, 0, s>>>(op, gp, g_stride, wp, outp, cols, eps);
  return cudaGetLastError();
}

template <typename T>
cudaError_t launch_clamped_glu(const void* gu, void* out, long long rows, int n, float limit, float alpha, float shift, cudaStream_t s) {
  if (rows == 0) return cudaSuccess;
  if (n % 8 == 0 && aligned16(gu) && aligned16(out))
    clamped_glu_kernel<T, 8><<<grid_1d(rows * (n / 8)), kThreads, 0, s>>>(static_cast<const T*>(gu), static_cast<T*>(out), rows, n,
                                                                         limit, alpha, shift);
  else
    clamped_glu_kernel<T, 1><<<grid_1d(rows * n), kThreads, 0, s>>>(static_cast<const T*>(gu), static_cast<T*>(out), rows, n, limit,
                                                                   alpha, shift);
  return cudaGetLastError();
}

template <typename T>
cudaError_t launch_side_gate(const void* z, const void* side, const int64_t* tokens, int vocab, long long side_stride, int off,
                             void* out, long long rows, int n, cudaStream_t s) {
  if (rows == 0) return cudaSuccess;
  const T *zp = static_cast<const T*>(z), *sp = static_cast<const T*>(side);
  T* op = static_cast<T*>(out);
  if (n % 8 == 0 && side_stride % 8 == 0 && off % 8 == 0 && aligned16(z) && aligned16(side) && aligned16(out))
    side_gate_kernel<T, 8><<<grid_1d(rows * (n / 8)), kThreads, 0, s>>>(zp, sp, tokens, vocab, side_stride, off, op, rows, n);
  else
    side_gate_kernel<T, 1><<<grid_1d(rows * n), kThreads, 0, s>>>(zp, sp, tokens, vocab, side_stride, off, op, rows, n);
  return cudaGetLastError();
}

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

#define FA_ROW_OPS(T)                                                                                                              \
  template cudaError_t launch_residual_norm<T>(const ResidualNormArgs&, cudaStream_t);                                            \
  template cudaError_t launch_gated_norm<T>(const void*, const void*, long long, const void*, void*, long long, int, float,       \
                                            cudaStream_t);                                                                        \
  template cudaError_t launch_clamped_glu<T>(const void*, void*, long long, int, float, float, float, cudaStream_t);              \
  template cudaError_t launch_side_gate<T>(const void*, const void*, const int64_t*, int, long long, int, void*, long long, int,  \
                                           cudaStream_t);                                                                         \
  template cudaError_t launch_latent_prep<T>(const LatentPrepArgs&, cudaStream_t);                                                \
  template cudaError_t launch_rotate_heads<T>(void*, const float*, const float*, long long, int, int, int, int, cudaStream_t);
FA_ROW_OPS(bf16)
FA_ROW_OPS(float)

}  // namespace hybrid
}  // namespace fa
