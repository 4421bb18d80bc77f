#include "kv_attention.cuh"
namespace fa { namespace mixers {
bool kv_decode_supported(const KvAttentionArgs&) { return false; }
int kv_decode_splits(long long, int, int, int, int) { return 1; }
cudaError_t launch_kv_decode(const KvAttentionArgs&, cudaStream_t) { return cudaErrorNotSupported; }
} }
