// Attention in the latent space, general kernel: any size, bfloat16 or float, sm_100a.
//
// The key of a cached token is its row (latent | rotated part), shared by all heads; the value is the latent itself.
// A query row is (q_unrotated W_uk | rotated part) and sees the keys 0 .. its position.  The result is the
// softmax-weighted latent, still to be multiplied by W_uv.
#include <math_constants.h>

#include "hybrid_common.cuh"
#include "latent_attention.cuh"

namespace fa {
namespace hybrid {
namespace {

constexpr int kTile = 128;     // keys per step = threads per CTA

template <typename T>
__global__ void __launch_bounds__(kTile) latent_attention_kernel(const LatentAttentionArgs a) {
  extern __shared__ float sm[];
  const int D = a.kv_rank + a.rot_dim;
  float* q = sm;                 // [D]
  float* acc = q + D;            // [kv_rank]
  float* p = acc + a.kv_rank;    // [kTile]
  float* red = p + kTile;        // [8]
  const T** rows = reinterpret_cast<const T**>(red + 8 + ((D + a.kv_rank) & 1));   // [kTile]
  const long long row = blockIdx.x;
  const int head = blockIdx.y, tid = threadIdx.x;
  const T* qa = static_cast<const T*>(a.q_abs) + (row * a.heads + head) * a.kv_rank;
  for (int c = tid; c < a.kv_rank; c += kTile) { q[c] = to_f(qa[c]) * a.scale; acc[c] = 0.f; }
  const int half = a.rot_dim / 2;
  const T* qr = static_cast<const T*>(a.q) + (row * a.heads + head) * a.q_stride + a.q_off;
  for (int i = tid; i < half; i += kTile) {
    const float cs = a.cos_t[row * half + i], sn = a.sin_t[row * half + i];
    const float u = to_f(qr[i]), v = to_f(qr[i + half]);
    q[a.kv_rank + i] = to_f(from_f<T>(u * cs - v * sn)) * a.scale;
    q[a.kv_rank + half + i] = to_f(from_f<T>(v * cs + u * sn)) * a.scale;
  }
  const int seq = a.tok_seq[row];
  int n = a.positions[row] + 1;
  bool bad = seq < 0 || seq >= a.n_seq || n <= 0 || (n + 15) / 16 > a.max_blocks;
  if (bad) n = 0;
  float m = -CUDART_INF_F, l = 0.f;
  for (int k0 = 0; k0 < n; k0 += kTile) {
    const int key = k0 + tid;
    const T* kr = nullptr;
    if (key < n) {
      const int page = a.block_table[(long long)seq * a.max_blocks + (key >> 4)];
      if (page >= 0 && page < a.n_blocks) kr = static_cast<const T*>(a.pool) + ((long long)page * 16 + (key & 15)) * a.pool_stride;
      else bad = true;
    }
    __syncthreads();             // q is complete; the previous step's p and rows are no longer read
    float s = -CUDART_INF_F;
    if (kr != nullptr) {
      s = 0.f;
      for (int c = 0; c < D; ++c) s += q[c] * to_f(kr[c]);
    }
    rows[tid] = kr;
    float mx = warp_max(s);
    if ((tid & 31) == 0) red[tid >> 5] = mx;
    __syncthreads();
    mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    const float m_new = fmaxf(m, mx);
    const float w = (kr != nullptr) ? expf(s - m_new) : 0.f;
    p[tid] = w;
    const float ws = warp_sum(w);
    if ((tid & 31) == 0) red[4 + (tid >> 5)] = ws;
    const float f = (m == -CUDART_INF_F) ? 0.f : expf(m - m_new);
    __syncthreads();
    l = l * f + red[4] + red[5] + red[6] + red[7];
    m = m_new;
    const int cnt = n - k0 < kTile ? n - k0 : kTile;
    for (int c = tid; c < a.kv_rank; c += kTile) {
      float o = acc[c] * f;
      for (int j = 0; j < cnt; ++j)
        if (rows[j] != nullptr) o += p[j] * to_f(rows[j][c]);
      acc[c] = o;
    }
  }
  __syncthreads();
  if (bad) atomicOr(a.status, 2);
  float g = l > 0.f ? 1.f / l : 0.f;
  if (a.gate != nullptr) g *= sigmoid_f(to_f(static_cast<const T*>(a.gate)[row * a.gate_stride + head]));
  T* out = static_cast<T*>(a.out) + (row * a.heads + head) * a.kv_rank;
  for (int c = tid; c < a.kv_rank; c += kTile) out[c] = from_f<T>(acc[c] * g);
}

}  // namespace

template <typename T>
cudaError_t launch_latent_attention(const LatentAttentionArgs& a, cudaStream_t s) {
  if (a.rows == 0) return cudaSuccess;
  const int D = a.kv_rank + a.rot_dim;
  const size_t smem = ((size_t)D + a.kv_rank + kTile + 8 + 1) * sizeof(float) + kTile * sizeof(void*);
  cudaError_t e = cudaFuncSetAttribute(latent_attention_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  latent_attention_kernel<T><<<dim3((unsigned)a.rows, (unsigned)a.heads), kTile, smem, s>>>(a);
  return cudaGetLastError();
}

template cudaError_t launch_latent_attention<bf16>(const LatentAttentionArgs&, cudaStream_t);
template cudaError_t launch_latent_attention<float>(const LatentAttentionArgs&, cudaStream_t);

}  // namespace hybrid
}  // namespace fa
