// Prompt attention inside chunks on the tcgen05 prefill kernel (prefill_tc5_kernel.cuh): a prompt cut at its chunks' borders is a
// batch of independent causal pieces, whose queries are the last keys of the piece; the distance bias goes to the scores as they
// are read from tensor memory, the element-wise gate to the output.
#include "../prefill_tc5_kernel.cuh"
#include "kv_attention.cuh"

namespace fa {
namespace mixers {
namespace {

template <int NA, int D>
cudaError_t launch_t(const KvPrefillArgs& a, EncodeTiledFn enc, cudaStream_t stream) {
  CUtensorMap qmap, kmap, vmap;
  const int H = a.heads, G = a.kv_heads;
  if (!make_map3(enc, &qmap, a.q, a.dim, H, a.total_q, a.dim, (long long)H * a.dim) ||
      !make_map3(enc, &kmap, a.k, a.dim, G, a.total_kv, a.dim, (long long)G * a.dim) ||
      !make_map3(enc, &vmap, a.v, a.vdim, G, a.total_kv, a.vdim, (long long)G * a.vdim))
    return cudaErrorInvalidValue;
  Tc5BiasParams p{};
  p.out = static_cast<__half*>(a.out);
  p.cu_seqlens = a.cu_q;
  p.cu_kv = a.cu_kv;
  p.total_kv = a.total_kv;
  p.status = a.status;
  p.bias = a.slopes;
  p.inv_scale = 1.f / a.scale;
  p.col_gate = static_cast<const __nv_bfloat16*>(a.gate);
  p.col_gate_stride = a.gate_stride;
  p.batch = a.n_piece;
  p.H_Q = H;
  p.H_KV = G;
  p.max_seqlen = a.max_q;
  p.total = a.total_q;
  p.o_head_stride = a.vdim;
  p.o_tok_stride = a.out_stride;
  p.causal = 1;
  p.D_real = a.vdim;
  p.pair_heads = (H / G) % 2 == 0;
  p.out_bf16 = 1;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  p.n_hg = p.pair_heads ? H / 2 : H;
  p.n_rb = p.pair_heads ? (a.max_q + 127) / 128 : (a.max_q + 255) / 256;
  const long long n_items = (long long)p.n_rb * p.batch * p.n_hg;
  int dev = 0, sms = 0;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  auto kern = prefill_tc5_kernel<NA, 0, D, 0, true, true>;
  constexpr int smem = Tc5Layout<NA, 0, D>::BYTES;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  e = next_item_counter(&p.item_counter, stream);
  if (e != cudaSuccess) return e;
  kern<<<dim3((unsigned)(n_items < sms ? n_items : sms)), 640, smem, stream>>>(qmap, kmap, vmap, qmap, kmap, p);
  return cudaGetLastError();
}

}  // namespace

bool kv_prefill_supported(int heads, int kv_heads, int dim, int vdim, float scale) {
  (void)heads; (void)kv_heads;
  return dim % 8 == 0 && vdim % 8 == 0 && dim <= 128 && vdim <= 128 && scale > 0.f;
}

cudaError_t launch_kv_prefill(const KvPrefillArgs& a, void* encode_fn, cudaStream_t s) {
  if (a.total_q == 0) return cudaSuccess;
  EncodeTiledFn enc = reinterpret_cast<EncodeTiledFn>(encode_fn);
  if (a.dim <= 64) return a.vdim <= 64 ? launch_t<1, 64>(a, enc, s) : launch_t<1, 128>(a, enc, s);
  return a.vdim <= 64 ? launch_t<2, 64>(a, enc, s) : launch_t<2, 128>(a, enc, s);
}

}  // namespace mixers
}  // namespace fa
