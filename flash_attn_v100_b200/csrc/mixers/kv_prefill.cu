#include "kv_attention.cuh"
namespace fa { namespace mixers {
bool kv_prefill_supported(int, int, int, int, float) { return false; }
cudaError_t launch_kv_prefill(const KvPrefillArgs&, void*, cudaStream_t) { return cudaErrorNotSupported; }
} }
