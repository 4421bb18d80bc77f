// Helpers shared by the hybrid decoder's kernels: element types, vector access, block reductions.
//
// Every kernel is built for two activation types: bfloat16 (serving) and float (full 32-bit).  Loads widen to fp32,
// arithmetic is fp32, stores round once.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace fa {
namespace hybrid {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

// N consecutive elements as fp32; N * sizeof(T) is 4, 8, 16 or 32 bytes and the address is aligned to
// min(16, N * sizeof(T)) when N > 1.
template <int N>
__device__ __forceinline__ void load_n(const float* p, float (&v)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N / 4; ++i) {
      const float4 a = reinterpret_cast<const float4*>(p)[i];
      v[4 * i] = a.x; v[4 * i + 1] = a.y; v[4 * i + 2] = a.z; v[4 * i + 3] = a.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = p[i];
  }
}
template <int N>
__device__ __forceinline__ void load_n(const bf16* p, float (&v)[N]) {
  if constexpr (N % 8 == 0) {
#pragma unroll
    for (int i = 0; i < N / 8; ++i) {
      union { uint4 u; bf16 h[8]; } a;
      a.u = reinterpret_cast<const uint4*>(p)[i];
#pragma unroll
      for (int j = 0; j < 8; ++j) v[8 * i + j] = to_f(a.h[j]);
    }
  } else if constexpr (N == 4) {
    union { uint2 u; bf16 h[4]; } a;
    a.u = *reinterpret_cast<const uint2*>(p);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = to_f(a.h[j]);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = to_f(p[i]);
  }
}
template <int N>
__device__ __forceinline__ void store_n(float* p, const float (&v)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N / 4; ++i)
      reinterpret_cast<float4*>(p)[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) p[i] = v[i];
  }
}
template <int N>
__device__ __forceinline__ void store_n(bf16* p, const float (&v)[N]) {
  if constexpr (N % 8 == 0) {
#pragma unroll
    for (int i = 0; i < N / 8; ++i) {
      union { uint4 u; bf16 h[8]; } a;
#pragma unroll
      for (int j = 0; j < 8; ++j) a.h[j] = from_f<bf16>(v[8 * i + j]);
      reinterpret_cast<uint4*>(p)[i] = a.u;
    }
  } else if constexpr (N == 4) {
    union { uint2 u; bf16 h[4]; } a;
#pragma unroll
    for (int j = 0; j < 4; ++j) a.h[j] = from_f<bf16>(v[j]);
    *reinterpret_cast<uint2*>(p) = a.u;
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) p[i] = from_f<bf16>(v[i]);
  }
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Sum over the block, in every thread; `red` holds one float per warp and is free again on return.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < (int)((blockDim.x + 31) >> 5); ++i) tot += red[i];
  __syncthreads();
  return tot;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z * sigmoid_f(z); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  const float c = 0.7978845608028654f;   // sqrt(2 / pi)
  return 0.5f * z * (1.f + tanhf(c * (z + 0.044715f * z * z * z)));
}

// The same for results that are rounded to T: with T = bfloat16 the hardware's exponential and reciprocal, whose errors are far below the
// rounding.  (Below -80 the sigmoid stays at its value there, 2e-35.)
template <typename T>
__device__ __forceinline__ float sigmoid_t(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-fmaxf(z, -80.f)));
  else return sigmoid_f(z);
}
template <typename T>
__device__ __forceinline__ float silu_t(float z) { return z * sigmoid_t<T>(z); }
template <typename T>
__device__ __forceinline__ float gelu_tanh_t(float z) {
  if constexpr (sizeof(T) == 2) {
    const float c2 = 2.f * 0.7978845608028654f;          // (1 + tanh(u)) / 2 = sigmoid(2 u)
    return z * sigmoid_t<T>(c2 * (z + 0.044715f * z * z * z));
  } else {
    return gelu_tanh_f(z);
  }
}

}  // namespace hybrid
}  // namespace fa
