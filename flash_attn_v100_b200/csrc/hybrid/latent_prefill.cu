// Prompt attention of the latent attention layers on the tcgen05 prefill kernel, and the gather of cached latent rows.
//
// For prompts the cached latents are expanded into per-head keys and values by one matrix product; the score is then an
// ordinary dot product over (dim unrotated | rot_dim rotated) columns, the rotated key columns being one row that all
// heads share.  The kernel is prefill_tc5_kernel.cuh with that shared part as a second pair of tensor maps (so it is never
// replicated per head in memory), keys of earlier passes (a sequence's queries are its last rows), and the head gate in
// the epilogue.
#include "../prefill_tc5_kernel.cuh"
#include "hybrid_common.cuh"
#include "latent_prefill.cuh"

namespace fa {
namespace hybrid {
namespace {

// One warp per (row, copy of 32 x 16 bytes): rows of the paged cache to contiguous rows.
template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentGatherArgs a) {
  const long long row = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (row >= a.total_kv) return;
  int lo = 0, hi = a.n_seq - 1;                 // last sequence that starts at or before the row
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (a.cu_kv[mid] <= row) lo = mid; else hi = mid - 1;
  }
  const int pos = (int)(row - a.cu_kv[lo]);
  int page = -1;
  if (pos >= 0 && (pos >> 4) < a.max_blocks) page = a.block_table[(long long)lo * a.max_blocks + (pos >> 4)];
  T* c = static_cast<T*>(a.c) + row * a.kv_rank;
  T* r = static_cast<T*>(a.r) + row * a.rot_dim;
  if (page < 0 || page >= a.n_blocks) {
    if (lane == 0) atomicOr(a.status, 2);
    for (int i = lane; i < a.kv_rank; i += 32) c[i] = from_f<T>(0.f);
    for (int i = lane; i < a.rot_dim; i += 32) r[i] = from_f<T>(0.f);
    return;
  }
  const T* src = static_cast<const T*>(a.pool) + ((long long)page * 16 + (pos & 15)) * a.pool_stride;
  constexpr int V = 16 / sizeof(T);
  if (a.kv_rank % V == 0 && a.rot_dim % V == 0) {
    for (int i = lane; i < a.kv_rank / V; i += 32) reinterpret_cast<uint4*>(c)[i] = reinterpret_cast<const uint4*>(src)[i];
    for (int i = lane; i < a.rot_dim / V; i += 32)
      reinterpret_cast<uint4*>(r)[i] = reinterpret_cast<const uint4*>(src + a.kv_rank)[i];
  } else {
    for (int i = lane; i < a.kv_rank; i += 32) c[i] = src[i];
    for (int i = lane; i < a.rot_dim; i += 32) r[i] = src[a.kv_rank + i];
  }
}

template <int NA, int D>
cudaError_t launch_t(const LatentPrefillArgs& a, EncodeTiledFn enc, cudaStream_t stream) {
  const auto* q = static_cast<const bf16*>(a.q);
  const auto* kv = static_cast<const bf16*>(a.kv);
  const int H = a.heads;
  const long long qs = a.dim + a.rot_dim, ks = (long long)H * (a.dim + a.vdim);
  CUtensorMap qmap, kmap, vmap, qmap_b, kmap_b;
  if (!make_map3(enc, &qmap, q, a.dim, H, a.total_q, qs, H * qs) ||
      !make_map3(enc, &qmap_b, q + a.dim, a.rot_dim, H, a.total_q, qs, H * qs) ||
      !make_map3(enc, &kmap, kv, a.dim, H, a.total_kv, a.dim, ks) ||
      !make_map3(enc, &vmap, kv + (long long)H * a.dim, a.vdim, H, a.total_kv, a.vdim, ks) ||
      !make_map3(enc, &kmap_b, a.kr, a.rot_dim, 1, a.total_kv, a.rot_dim, a.rot_dim))
    return cudaErrorInvalidValue;
  Tc5SharedParams p{};
  p.out = static_cast<__half*>(a.out);
  p.cu_seqlens = a.cu_q;
  p.cu_kv = a.cu_kv;
  p.total_kv = a.total_kv;
  p.gate = static_cast<const bf16*>(a.gate);
  p.gate_stride = a.gate_stride;
  p.status = a.status;
  p.batch = a.n_seq;
  p.H_Q = p.H_KV = H;
  p.max_seqlen = a.max_q;
  p.total = a.total_q;
  p.o_head_stride = a.vdim;
  p.o_tok_stride = (long long)H * a.vdim;
  p.causal = 1;
  p.D_real = a.vdim;
  p.pair_heads = 0;            // every head has keys of its own: the two tiles are row blocks of one head
  p.out_bf16 = 1;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  p.n_hg = H;
  p.n_rb = (a.max_q + 255) / 256;
  const long long n_items = (long long)p.n_rb * p.batch * p.n_hg;
  int dev = 0, sms = 0;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  auto kern = prefill_tc5_kernel<NA, 1, D, 0, true>;
  constexpr int smem = Tc5Layout<NA, 1, D>::BYTES;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  e = next_item_counter(&p.item_counter, stream);
  if (e != cudaSuccess) return e;
  kern<<<dim3((unsigned)(n_items < sms ? n_items : sms)), 640, smem, stream>>>(qmap, kmap, vmap, qmap_b, kmap_b, p);
  return cudaGetLastError();
}

}  // namespace

bool latent_prefill_supported(int dim, int rot_dim, int vdim, float scale) {
  return dim % 8 == 0 && rot_dim % 8 == 0 && vdim % 8 == 0 && dim > 0 && dim <= 128 && rot_dim > 0 && rot_dim <= 64 && vdim > 0 &&
         vdim <= 128 && scale > 0.f;
}

cudaError_t launch_latent_prefill(const LatentPrefillArgs& a, void* encode_fn, cudaStream_t s) {
  if (a.total_q == 0) return cudaSuccess;
  EncodeTiledFn enc = reinterpret_cast<EncodeTiledFn>(encode_fn);
  if (a.dim <= 64) return a.vdim <= 64 ? launch_t<1, 64>(a, enc, s) : launch_t<1, 128>(a, enc, s);
  return a.vdim <= 64 ? launch_t<2, 64>(a, enc, s) : launch_t<2, 128>(a, enc, s);
}

template <typename T>
cudaError_t launch_latent_gather(const LatentGatherArgs& a, cudaStream_t s) {
  if (a.total_kv == 0) return cudaSuccess;
  latent_gather_kernel<T><<<(unsigned)((a.total_kv + 7) / 8), 256, 0, s>>>(a);
  return cudaGetLastError();
}
template cudaError_t launch_latent_gather<bf16>(const LatentGatherArgs&, cudaStream_t);
template cudaError_t launch_latent_gather<float>(const LatentGatherArgs&, cudaStream_t);

}  // namespace hybrid
}  // namespace fa
