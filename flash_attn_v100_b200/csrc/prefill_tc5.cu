// Launcher of the tcgen05 prefill kernel (prefill_tc5_kernel.cuh) for the dense and packed attention operators.
#include "prefill.cuh"
#include "prefill_tc5_kernel.cuh"

namespace fa {

namespace {

bool g_tc5_poly = false;  // true: a quarter of the exponentials evaluated as a polynomial on the FMA pipes

using Tc5Kernel = void (*)(const CUtensorMap, const CUtensorMap, const CUtensorMap, const CUtensorMap, const CUtensorMap, const Tc5Params);

template <int D>
Tc5Kernel pick_kernel() {
  return g_tc5_poly ? prefill_tc5_kernel<D / 64, 0, D, 2, false> : prefill_tc5_kernel<D / 64, 0, D, 0, false>;
}
template <int D>
Tc5Kernel pick_kernel_bf16() {
  return g_tc5_poly ? prefill_tc5_kernel<D / 64, 0, D, 2, true> : prefill_tc5_kernel<D / 64, 0, D, 0, true>;
}

template <int D>
cudaError_t launch_tc5_t(const PrefillParams& pp, void* encode_fn, cudaStream_t stream) {
  EncodeTiledFn enc = reinterpret_cast<EncodeTiledFn>(encode_fn);
  const bool dense = pp.cu_seqlens == nullptr;
  CUtensorMap qmap, kmap, vmap;
  bool ok;
  if (dense) {
    const long long qrows = (long long)pp.batch * pp.H_Q * pp.N, krows = (long long)pp.batch * pp.H_KV * pp.N;
    const int Dr = pp.D_real;   // extent of the innermost dimension: the boxes' columns past it are zero-filled
    ok = make_map3(enc, &qmap, pp.q, Dr, 1, qrows, Dr, Dr) && make_map3(enc, &kmap, pp.k, Dr, 1, krows, Dr, Dr) &&
         make_map3(enc, &vmap, pp.v, Dr, 1, krows, Dr, Dr);
  } else {
    const int Dr = pp.D_real;
    ok = make_map3(enc, &qmap, pp.q, Dr, pp.H_Q, pp.total, Dr, (long long)pp.H_Q * Dr) &&
         make_map3(enc, &kmap, pp.k, Dr, pp.H_KV, pp.total, Dr, (long long)pp.H_KV * Dr) &&
         make_map3(enc, &vmap, pp.v, Dr, pp.H_KV, pp.total, Dr, (long long)pp.H_KV * Dr);
  }
  if (!ok) return cudaErrorInvalidValue;
  Tc5Params p{};
  p.out = pp.out;
  p.cu_seqlens = pp.cu_seqlens;
  p.batch = pp.batch; p.H_Q = pp.H_Q; p.H_KV = pp.H_KV; p.N = pp.N; p.max_seqlen = pp.max_seqlen;
  p.total = pp.total;
  p.o_batch_stride = pp.q_batch_stride; p.o_head_stride = pp.q_head_stride; p.o_tok_stride = pp.q_tok_stride;
  p.causal = pp.causal;
  p.D_real = pp.D_real;
  p.pair_heads = ((pp.H_Q / pp.H_KV) % 2 == 0) ? 1 : 0;
  p.dense = dense ? 1 : 0;
  p.out_bf16 = (pp.out_bf16 || pp.in_bf16) ? 1 : 0;
  p.scale_log2 = pp.scale_log2;
  const size_t smem = Tc5Layout<D / 64, 0, D>::BYTES;
  Tc5Kernel kern = pp.in_bf16 ? pick_kernel_bf16<D>() : pick_kernel<D>();
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  const int max_len = dense ? pp.N : pp.max_seqlen;
  dim3 grid;
  if (p.pair_heads) { p.n_hg = pp.H_Q / 2; p.n_rb = (max_len + 127) / 128; }
  else { p.n_hg = pp.H_Q; p.n_rb = (max_len + 255) / 256; }
  const long long n_items = (long long)p.n_rb * pp.batch * p.n_hg;
  int dev = 0, sms = 0;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  grid = dim3((unsigned)(n_items < sms ? n_items : sms));
  e = next_item_counter(&p.item_counter, stream);
  if (e != cudaSuccess) return e;
  kern<<<grid, 640, smem, stream>>>(qmap, kmap, vmap, qmap, kmap, p);
  return cudaGetLastError();
}

}  // namespace

bool prefill_tc5_supported(const PrefillParams& p, int D) {
  if (D != 64 && D != 128) return false;
  const long long qrows = p.cu_seqlens ? p.total : (long long)p.batch * p.H_Q * p.N;
  if (qrows >= (1ll << 31)) return false;
  return true;
}

cudaError_t launch_prefill_tc5(const PrefillParams& p, int D, void* encode_fn, cudaStream_t stream) {
  if (D == 128) return launch_tc5_t<128>(p, encode_fn, stream);
  if (D == 64) return launch_tc5_t<64>(p, encode_fn, stream);
  return cudaErrorInvalidValue;
}

#ifdef FA_TC5_PROF
// Instrumented build only: copy the wait counters to the host (and optionally clear them).
extern "C" int fa_debug_read_tc5_prof(unsigned long long* host, int clear) {
  cudaError_t e = cudaMemcpyFromSymbol(host, g_tc5_prof, sizeof(unsigned long long) * 5 * 16);
  if (e == cudaSuccess && clear) {
    static const unsigned long long zeros[5 * 16] = {0};
    e = cudaMemcpyToSymbol(g_tc5_prof, zeros, sizeof(zeros));
  }
  return (int)e;
}
#endif

void prefill_tc5_set_poly(bool on) { g_tc5_poly = on; }

cudaError_t prefill_status_ptr(int** out) {
  void* ptr = nullptr;
  cudaError_t e = cudaGetSymbolAddress(&ptr, g_prefill_status);
  *out = static_cast<int*>(ptr);
  return e;
}

cudaError_t prefill_status(int* host_out, cudaStream_t stream) {
  cudaError_t e = cudaMemcpyFromSymbolAsync(host_out, g_prefill_status, sizeof(int), 0, cudaMemcpyDeviceToHost, stream);
  if (e != cudaSuccess) return e;
  return cudaStreamSynchronize(stream);
}

cudaError_t prefill_status_clear(cudaStream_t stream) {
  int zero = 0;
  return cudaMemcpyToSymbolAsync(g_prefill_status, &zero, sizeof(int), 0, cudaMemcpyHostToDevice, stream);
}

}  // namespace fa
