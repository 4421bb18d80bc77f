// Decayed linear attention, token by token: S <- d S + k v^T, o = S^T q, with SiLU on q, k and v, sm_100a.
//
// q, k and v are read from the fused projection's rows and activated on the way in; the state S [dk, dv] of every head
// is fp32 and lives in a slot of the cache between calls.  A sequence whose first token is at position 0 starts from
// zero whatever its slot holds.
#include "hybrid_common.cuh"
#include "lightning.cuh"

namespace fa {
namespace hybrid {
namespace {

constexpr int kCols = 32;      // value columns per CTA of the scan kernel
constexpr int kRowGroups = 8;

// Sequence `seq`: its tokens [t0, t0 + n) and its state (null if the slot is not one of the cache's).
__device__ __forceinline__ float* locate(const LightningArgs& a, int seq, int head, long long& t0, int& n) {
  if (a.cu != nullptr) {
    t0 = a.cu[seq];
    long long e = a.cu[seq + 1];
    if (t0 < 0) t0 = 0;
    if (e > a.total) e = a.total;
    n = e > t0 ? (int)(e - t0) : 0;
  } else {
    t0 = seq;
    n = 1;
  }
  const int slot = a.slots[seq];
  if (slot < 0 || slot >= a.n_slots) {
    if (threadIdx.x == 0) atomicOr(a.status, 2);
    return nullptr;
  }
  return a.state + ((long long)slot * a.heads + head) * a.dk * a.dv;
}

template <typename T>
__global__ void __launch_bounds__(kCols * kRowGroups) lightning_scan_kernel(const LightningArgs a) {
  extern __shared__ float sm[];
  float* S = sm;                          // [dk][kCols]
  float* sq = S + a.dk * kCols;           // [dk]
  float* sk = sq + a.dk;                  // [dk]
  float* red = sk + a.dk;                 // [kRowGroups][kCols]
  const int seq = blockIdx.x, head = blockIdx.y, c0 = blockIdx.z * kCols;
  const int lane = threadIdx.x & 31, rg = threadIdx.x >> 5;
  const int col = c0 + lane;
  const bool live = col < a.dv;
  long long t0;
  int n;
  float* state = locate(a, seq, head, t0, n);
  if (n == 0) return;
  const bool fresh = a.starts[seq] == 0;
  for (int r = rg; r < a.dk; r += kRowGroups)
    S[r * kCols + lane] = (!fresh && live && state) ? state[(long long)r * a.dv + col] : 0.f;
  const float d = a.decay[head];
  const T* base = static_cast<const T*>(a.qkv);
  T* out = static_cast<T*>(a.out);
  for (int t = 0; t < n; ++t) {
    const T* row = base + (t0 + t) * a.stride;
    __syncthreads();
    for (int i = threadIdx.x; i < a.dk; i += blockDim.x) {
      sq[i] = to_f(from_f<T>(silu_f(to_f(row[a.off_q + head * a.dk + i]))));
      sk[i] = to_f(from_f<T>(silu_f(to_f(row[a.off_k + head * a.dk + i]))));
    }
    const float v = live ? to_f(from_f<T>(silu_f(to_f(row[a.off_v + head * a.dv + col])))) : 0.f;
    __syncthreads();
    float o = 0.f;
    for (int r = rg; r < a.dk; r += kRowGroups) {
      const float s = d * S[r * kCols + lane] + sk[r] * v;
      S[r * kCols + lane] = s;
      o += sq[r] * s;
    }
    red[rg * kCols + lane] = o;
    __syncthreads();
    if (rg == 0 && live) {
#pragma unroll
      for (int i = 1; i < kRowGroups; ++i) o += red[i * kCols + lane];
      out[(t0 + t) * (long long)a.heads * a.dv + (long long)head * a.dv + col] = from_f<T>(o);
    }
  }
  if (state && live)
    for (int r = rg; r < a.dk; r += kRowGroups) state[(long long)r * a.dv + col] = S[r * kCols + lane];
}

// One token per sequence.  CTA = (sequence, head, range of value columns); a thread owns four columns of every n_rg-th
// state row, so the state is read and written once with 16-byte accesses.
template <typename T>
__global__ void __launch_bounds__(256) lightning_decode_kernel(const LightningArgs a, const int cols) {
  extern __shared__ float sm[];
  float* sq = sm;                         // [dk]
  float* sk = sq + a.dk;                  // [dk]
  float* red = sk + a.dk;                 // [n_rg][cols]
  const int seq = blockIdx.x, head = blockIdx.y, c0 = blockIdx.z * cols;
  const int my_cols = min(cols, a.dv - c0);
  const int n4 = cols / 4, n_rg = blockDim.x / n4;
  const int cg = threadIdx.x % n4, rg = threadIdx.x / n4;
  long long t0;
  int n;
  float* state = locate(a, seq, head, t0, n);
  if (state == nullptr) return;           // (uniform over the CTA)
  const bool fresh = a.starts[seq] == 0;
  const T* row = static_cast<const T*>(a.qkv) + t0 * a.stride;
  const bool live = rg < n_rg && cg * 4 < my_cols;
  float v[4] = {0.f, 0.f, 0.f, 0.f};
  if (live) {
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = to_f(from_f<T>(silu_f(to_f(row[a.off_v + head * a.dv + c0 + cg * 4 + j]))));
  }
  for (int i = threadIdx.x; i < a.dk; i += blockDim.x) {
    sq[i] = to_f(from_f<T>(silu_f(to_f(row[a.off_q + head * a.dk + i]))));
    sk[i] = to_f(from_f<T>(silu_f(to_f(row[a.off_k + head * a.dk + i]))));
  }
  __syncthreads();
  const float d = a.decay[head];
  float o[4] = {0.f, 0.f, 0.f, 0.f};
  if (live) {
    float* sp = state + c0 + cg * 4;
    int r = rg;
    constexpr int U = 8;
    for (; r + (U - 1) * n_rg < a.dk; r += U * n_rg) {
      float4 s[U];
#pragma unroll
      for (int u = 0; u < U; ++u)
        s[u] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(sp + (long long)(r + u * n_rg) * a.dv);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const float k = sk[r + u * n_rg], q = sq[r + u * n_rg];
        s[u].x = d * s[u].x + k * v[0]; s[u].y = d * s[u].y + k * v[1];
        s[u].z = d * s[u].z + k * v[2]; s[u].w = d * s[u].w + k * v[3];
        *reinterpret_cast<float4*>(sp + (long long)(r + u * n_rg) * a.dv) = s[u];
        o[0] += q * s[u].x; o[1] += q * s[u].y; o[2] += q * s[u].z; o[3] += q * s[u].w;
      }
    }
    for (; r < a.dk; r += n_rg) {
      float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(sp + (long long)r * a.dv);
      const float k = sk[r], q = sq[r];
      s.x = d * s.x + k * v[0]; s.y = d * s.y + k * v[1]; s.z = d * s.z + k * v[2]; s.w = d * s.w + k * v[3];
      *reinterpret_cast<float4*>(sp + (long long)r * a.dv) = s;
      o[0] += q * s.x; o[1] += q * s.y; o[2] += q * s.z; o[3] += q * s.w;
    }
  }
  if (rg < n_rg) {
#pragma unroll
    for (int j = 0; j < 4; ++j) red[rg * cols + cg * 4 + j] = o[j];
  }
  __syncthreads();
  T* out = static_cast<T*>(a.out) + t0 * (long long)a.heads * a.dv + (long long)head * a.dv + c0;
  for (int c = threadIdx.x; c < my_cols; c += blockDim.x) {
    float acc = 0.f;
    for (int i = 0; i < n_rg; ++i) acc += red[i * cols + c];
    out[c] = from_f<T>(acc);
  }
}

}  // namespace

template <typename T>
cudaError_t launch_lightning_scan(const LightningArgs& a, cudaStream_t s) {
  if (a.n_seq == 0) return cudaSuccess;
  const size_t smem = ((size_t)a.dk * (kCols + 2) + kRowGroups * kCols) * sizeof(float);
  cudaError_t e = cudaFuncSetAttribute(lightning_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  dim3 grid((unsigned)a.n_seq, (unsigned)a.heads, (unsigned)((a.dv + kCols - 1) / kCols));
  lightning_scan_kernel<T><<<grid, kCols * kRowGroups, smem, s>>>(a);
  return cudaGetLastError();
}

bool lightning_decode_supported(const LightningArgs& a) {
  return a.cu == nullptr && a.dv % 4 == 0 && a.dv <= 1024 && a.dk <= 2048 && (reinterpret_cast<uintptr_t>(a.state) & 15) == 0;
}

template <typename T>
cudaError_t launch_lightning_decode(const LightningArgs& a, int sm_count, cudaStream_t s) {
  if (a.n_seq == 0) return cudaSuccess;
  // value columns per CTA: the whole head, or a part of it while that leaves SMs without work
  int cols = (a.dv + 31) / 32 * 32;
  while (cols > 32 && (long long)a.n_seq * a.heads * ((a.dv + cols - 1) / cols) < 2ll * sm_count) cols = (cols / 2 + 31) / 32 * 32;
  const int n_rg = 256 / (cols / 4);
  const size_t smem = ((size_t)2 * a.dk + (size_t)n_rg * cols) * sizeof(float);
  dim3 grid((unsigned)a.n_seq, (unsigned)a.heads, (unsigned)((a.dv + cols - 1) / cols));
  lightning_decode_kernel<T><<<grid, 256, smem, s>>>(a, cols);
  return cudaGetLastError();
}

template cudaError_t launch_lightning_scan<bf16>(const LightningArgs&, cudaStream_t);
template cudaError_t launch_lightning_scan<float>(const LightningArgs&, cudaStream_t);
template cudaError_t launch_lightning_decode<bf16>(const LightningArgs&, int, cudaStream_t);
template cudaError_t launch_lightning_decode<float>(const LightningArgs&, int, cudaStream_t);

}  // namespace hybrid
}  // namespace fa
