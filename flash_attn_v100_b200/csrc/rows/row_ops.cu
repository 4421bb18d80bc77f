// Row-wise operators of the hybrid decoders, sm_100a: residual update + RMS norm (one or two weights), gated output norms,
// feed-forward activations, token side input, rows of the bigram embedding.
//
// The residual stream is fp32; activations are T (bfloat16 or float).  Every operator is one pass over its rows
// (HBM-bound); the vector width is chosen at launch from the sizes, so that any width runs.
#include "../hybrid/hybrid_common.cuh"
#include "row_ops.cuh"

namespace fa {
namespace hybrid {
namespace {

constexpr int kThreads = 256;

// KEEP: vectors per thread that stay in registers between the passes over a row (0: the row is read again).
// x (+)= [embedding] + [delta or rmsnorm(delta) * delta_w]; out = rmsnorm(x) * w (or x), out2 = rmsnorm(x) * w2.  One CTA per
// row.  MORE: further embedding tables are added to the embedding (embed_mode 2).
template <typename T, int VEC, int KEEP, bool MORE>
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
  const T* more[2] = {nullptr, nullptr};
  if constexpr (MORE) {
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      if (a.more[k] == nullptr) continue;
      int r = a.more_rows[k][row];
      r = r < 0 ? 0 : (r >= a.more_n[k] ? a.more_n[k] - 1 : r);
      more[k] = static_cast<const T*>(a.more[k]) + (long long)r * a.cols;
    }
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
      if constexpr (MORE) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] *= a.embed_scale;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          if (more[k] == nullptr) continue;
          float t[VEC];
          load_n<VEC>(more[k] + c * VEC, t);
#pragma unroll
          for (int i = 0; i < VEC; ++i) v[i] += t[i];
        }
      }
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
  T* out2 = a.out2 != nullptr ? static_cast<T*>(a.out2) + row * a.cols : nullptr;
  auto emit = [&](int c, float (&v)[VEC]) {
    if (out2 != nullptr) {
      float wv[VEC];
      load_n<VEC>(static_cast<const T*>(a.w2) + c * VEC, wv);
#pragma unroll
      for (int i = 0; i < VEC; ++i) wv[i] = v[i] * inv * wv[i];
      store_n<VEC>(out2 + c * VEC, wv);
    }
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

// Gated norm of row `blockIdx.x`, part `blockIdx.y` of `a.group` columns, one CTA each.  SILU: out = rmsnorm(o * silu(g)) * w,
// otherwise out = rmsnorm(o) * w * sigmoid(g).
template <typename T, bool SILU>
__device__ __forceinline__ float gate_first(float o, float g) { return SILU ? o * silu_t<T>(g) : o; }
template <typename T, bool SILU>
__device__ __forceinline__ float gate_last(float y, float g) { return SILU ? y : y * sigmoid_t<T>(g); }

template <typename T, int VEC, int KEEP, bool SILU>
__global__ void __launch_bounds__(kThreads) gated_norm_kernel(const GatedNormArgs a) {
  __shared__ float red[kThreads / 32];
  const long long row = blockIdx.x;
  const long long c0 = (long long)blockIdx.y * a.group;
  const T* o = static_cast<const T*>(a.o) + row * a.cols + c0;
  const T* g = static_cast<const T*>(a.g) + row * a.g_stride + c0;
  const T* w = static_cast<const T*>(a.w) + c0;
  T* out = static_cast<T*>(a.out) + row * a.out_stride + c0;
  const int nv = a.group / VEC;
  float keep[KEEP > 0 ? KEEP : 1][VEC];
  float ss = 0.f;
  auto fetch = [&](int c, float (&v)[VEC]) {
    load_n<VEC>(o + c * VEC, v);
    if constexpr (SILU) {
      float gv[VEC];
      load_n<VEC>(g + c * VEC, gv);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = gate_first<T, SILU>(v[i], gv[i]);
    }
  };
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int n = 0; n < KEEP; ++n) {
      const int c = threadIdx.x + n * kThreads;
      if (c < nv) {
        fetch(c, keep[n]);
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss += keep[n][i] * keep[n][i];
      }
    }
  } else {
    for (int c = threadIdx.x; c < nv; c += kThreads) {
      fetch(c, keep[0]);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss += keep[0][i] * keep[0][i];
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)a.group + a.eps);
  auto emit = [&](int c, float (&v)[VEC]) {
    float wv[VEC], gv[VEC];
    load_n<VEC>(w + c * VEC, wv);
    if constexpr (!SILU) load_n<VEC>(g + c * VEC, gv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = gate_last<T, SILU>(v[i] * inv * wv[i], SILU ? 0.f : gv[i]);
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
      fetch(c, keep[0]);
      emit(c, keep[0]);
    }
  }
}

// The same for parts of at most LANES * KEEP * 8 columns (a multiple of 8): LANES lanes per (row, part), KEEP vectors each.
template <typename T, int LANES, int KEEP, bool SILU>
__global__ void __launch_bounds__(kThreads) gated_norm_small_kernel(const GatedNormArgs a, const long long parts) {
  constexpr int VEC = 8;
  const long long part = ((long long)blockIdx.x * kThreads + threadIdx.x) / LANES;
  const int lane = threadIdx.x % LANES;
  const int per_row = a.cols / a.group;
  const bool live = part < parts;
  const long long row = live ? part / per_row : 0;
  const int c0 = live ? (int)(part - row * per_row) * a.group : 0;
  const T* o = static_cast<const T*>(a.o) + row * a.cols + c0;
  const T* g = static_cast<const T*>(a.g) + row * a.g_stride + c0;
  float v[KEEP][VEC], gv[KEEP][VEC];
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < KEEP; ++n) {
    const int c = (lane + n * LANES) * VEC;
    if (live && c < a.group) {
      load_n<VEC>(o + c, v[n]);
      load_n<VEC>(g + c, gv[n]);
    }
  }
#pragma unroll
  for (int n = 0; n < KEEP; ++n) {
    if (live && (lane + n * LANES) * VEC < a.group) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        v[n][i] = gate_first<T, SILU>(v[n][i], gv[n][i]);
        ss += v[n][i] * v[n][i];
      }
    }
  }
#pragma unroll
  for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!live) return;
  const float inv = 1.f / sqrtf(ss / (float)a.group + a.eps);
#pragma unroll
  for (int n = 0; n < KEEP; ++n) {
    const int c = (lane + n * LANES) * VEC;
    if (c >= a.group) break;
    float wv[VEC];
    load_n<VEC>(static_cast<const T*>(a.w) + c0 + c, wv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[n][i] = gate_last<T, SILU>(v[n][i] * inv * wv[i], gv[n][i]);
    store_n<VEC>(static_cast<T*>(a.out) + row * a.out_stride + c0 + c, v[n]);
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

// out = gelu_tanh(z), rows of n elements with any strides
template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads) gelu_kernel(const T* z, long long z_stride, T* out, long long out_stride, long long rows, int n) {
  const int nv = n / VEC;
  const long long total = rows * nv;
  for (long long i = (long long)blockIdx.x * kThreads + threadIdx.x; i < total; i += (long long)gridDim.x * kThreads) {
    const long long row = i / nv;
    const int c = (int)(i - row * nv) * VEC;
    float v[VEC];
    load_n<VEC>(z + row * z_stride + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = gelu_tanh_t<T>(v[j]);
    store_n<VEC>(out + row * out_stride + c, v);
  }
}

// Row of a bigram table for every token: (previous token * mul_prev + token * mul_cur) mod buckets, `buckets` for a sequence's
// first token.  The last token of the call is kept in the sequence's slot of `last`.  One CTA per sequence.
__global__ void __launch_bounds__(kThreads) bigram_rows_kernel(const int64_t* tokens, const int32_t* cu, const int32_t* starts,
                                                              const int32_t* slots, int32_t* last, int n_slots, long long total,
                                                              long long buckets, long long mul_prev, long long mul_cur,
                                                              int32_t* out, int* status) {
  const int seq = blockIdx.x;
  long long t0 = seq, t1 = seq + 1;
  if (cu != nullptr) {
    t0 = cu[seq];
    t1 = cu[seq + 1];
  }
  if (t0 < 0) t0 = 0;
  if (t1 > total) t1 = total;
  const int slot = slots[seq];
  const bool ok = slot >= 0 && slot < n_slots;
  if (!ok && threadIdx.x == 0) atomicOr(status, 2);
  const bool fresh = starts[seq] == 0;
  for (long long t = t0 + threadIdx.x; t < t1; t += kThreads) {
    long long prev = 0;
    bool first = false;
    if (t > t0) prev = tokens[t - 1];
    else if (fresh) first = true;
    else prev = ok ? last[slot] : 0;
    out[t] = (int32_t)(first ? buckets : (prev * mul_prev + (long long)tokens[t] * mul_cur) % buckets);
  }
  __syncthreads();
  if (threadIdx.x == 0 && ok && t1 > t0) last[slot] = (int32_t)tokens[t1 - 1];
}

unsigned grid_1d(long long threads) {
  long long blocks = (threads + kThreads - 1) / kThreads;
  if (blocks > 148 * 32) blocks = 148 * 32;
  return (unsigned)(blocks < 1 ? 1 : blocks);
}
bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

template <typename T, bool MORE>
static void launch_residual_norm_t(const ResidualNormArgs& a, bool vec, cudaStream_t s) {
  const unsigned g = (unsigned)a.rows;
  if (vec && a.cols <= 4 * kThreads) residual_norm_kernel<T, 4, 1, MORE><<<g, kThreads, 0, s>>>(a);
  else if (vec && a.cols <= 16 * kThreads) residual_norm_kernel<T, 4, 4, MORE><<<g, kThreads, 0, s>>>(a);
  else if (vec && a.cols <= 32 * kThreads) residual_norm_kernel<T, 4, 8, MORE><<<g, kThreads, 0, s>>>(a);
  else if (vec) residual_norm_kernel<T, 4, 0, MORE><<<g, kThreads, 0, s>>>(a);
  else residual_norm_kernel<T, 1, 0, MORE><<<g, kThreads, 0, s>>>(a);
}

template <typename T>
cudaError_t launch_residual_norm(const ResidualNormArgs& a, cudaStream_t s) {
  if (a.rows == 0) return cudaSuccess;
  const bool vec = a.cols % 4 == 0 && aligned16(a.x) && aligned16(a.delta) && aligned16(a.delta_w) && aligned16(a.embed) &&
                   aligned16(a.w) && aligned16(a.out) && aligned16(a.w2) && aligned16(a.out2) && aligned16(a.more[0]) && aligned16(a.more[1]);
  if (a.more[0] != nullptr || a.more[1] != nullptr || a.embed_scale != 1.f) launch_residual_norm_t<T, true>(a, vec, s);
  else launch_residual_norm_t<T, false>(a, vec, s);
  return cudaGetLastError();
}

template <typename T, bool SILU>
static void launch_gated_norm_t(const GatedNormArgs& a, cudaStream_t s) {
  const bool vec = a.group % 8 == 0 && a.g_stride % 8 == 0 && a.out_stride % 8 == 0 && aligned16(a.o) && aligned16(a.g) && aligned16(a.w) &&
                   aligned16(a.out);
  const dim3 grid((unsigned)a.rows, (unsigned)(a.cols / a.group));
  const long long parts = a.rows * (a.cols / a.group);
  auto blocks = [&](int lanes) { return (unsigned)((parts * lanes + kThreads - 1) / kThreads); };
  if (vec && a.group <= 64) gated_norm_small_kernel<T, 8, 1, SILU><<<blocks(8), kThreads, 0, s>>>(a, parts);
  else if (vec && a.group <= 128) gated_norm_small_kernel<T, 8, 2, SILU><<<blocks(8), kThreads, 0, s>>>(a, parts);
  else if (vec && a.group <= 256) gated_norm_small_kernel<T, 16, 2, SILU><<<blocks(16), kThreads, 0, s>>>(a, parts);
  else if (vec && a.group <= 512) gated_norm_small_kernel<T, 32, 2, SILU><<<blocks(32), kThreads, 0, s>>>(a, parts);
  else if (vec && a.group <= 1024) gated_norm_small_kernel<T, 32, 4, SILU><<<blocks(32), kThreads, 0, s>>>(a, parts);
  else if (vec && a.group <= 8 * kThreads) gated_norm_kernel<T, 8, 1, SILU><<<grid, kThreads, 0, s>>>(a);
  else if (vec && a.group <= 16 * kThreads) gated_norm_kernel<T, 8, 2, SILU><<<grid, kThreads, 0, s>>>(a);
  else if (vec && a.group <= 32 * kThreads) gated_norm_kernel<T, 8, 4, SILU><<<grid, kThreads, 0, s>>>(a);
  else if (vec) gated_norm_kernel<T, 8, 0, SILU><<<grid, kThreads, 0, s>>>(a);
  else gated_norm_kernel<T, 1, 0, SILU><<<grid, kThreads, 0, s>>>(a);
}

template <typename T>
cudaError_t launch_gated_norm(const GatedNormArgs& a, cudaStream_t s) {
  if (a.rows == 0) return cudaSuccess;
  if (a.silu_first) launch_gated_norm_t<T, true>(a, s);
  else launch_gated_norm_t<T, false>(a, s);
  return cudaGetLastError();
}

template <typename T>
cudaError_t launch_gelu(const void* z, long long z_stride, void* out, long long out_stride, long long rows, int n, cudaStream_t s) {
  if (rows == 0) return cudaSuccess;
  const T* zp = static_cast<const T*>(z);
  T* op = static_cast<T*>(out);
  if (n % 8 == 0 && z_stride % 8 == 0 && out_stride % 8 == 0 && aligned16(z) && aligned16(out))
    gelu_kernel<T, 8><<<grid_1d(rows * (n / 8)), kThreads, 0, s>>>(zp, z_stride, op, out_stride, rows, n);
  else
    gelu_kernel<T, 1><<<grid_1d(rows * n), kThreads, 0, s>>>(zp, z_stride, op, out_stride, rows, n);
  return cudaGetLastError();
}

cudaError_t launch_bigram_rows(const int64_t* tokens, const int32_t* cu, const int32_t* starts, const int32_t* slots, int32_t* last, int n_slots,
                               int n_seq, long long total, long long buckets, long long mul_prev, long long mul_cur, int32_t* out, int* status,
                               cudaStream_t s) {
  if (n_seq == 0) return cudaSuccess;
  bigram_rows_kernel<<<(unsigned)n_seq, kThreads, 0, s>>>(tokens, cu, starts, slots, last, n_slots, total, buckets, mul_prev, mul_cur, out, status);
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

#define FA_ROW_OPS(T)                                                                                                              \
  template cudaError_t launch_residual_norm<T>(const ResidualNormArgs&, cudaStream_t);                                            \
  template cudaError_t launch_gated_norm<T>(const GatedNormArgs&, cudaStream_t);                                                  \
  template cudaError_t launch_gelu<T>(const void*, long long, void*, long long, long long, int, cudaStream_t);                    \
  template cudaError_t launch_clamped_glu<T>(const void*, void*, long long, int, float, float, float, cudaStream_t);              \
  template cudaError_t launch_side_gate<T>(const void*, const void*, const int64_t*, int, long long, int, void*, long long, int,  \
                                           cudaStream_t);
FA_ROW_OPS(bf16)
FA_ROW_OPS(float)

}  // namespace hybrid
}  // namespace fa
