// What the C ABIs of the decoder libraries share: error texts, argument checks, device queries.  One per library: everything
// has internal linkage.
#pragma once
#include <cuda_runtime.h>
#include <stdarg.h>
#include <stdint.h>
#include <stdio.h>

namespace {

constexpr int FA_ABI_OK = 0, FA_ABI_ERR_INVALID_ARGUMENT = -1, FA_ABI_ERR_UNSUPPORTED = -2, FA_ABI_ERR_CUDA = -4;   // as in the headers
constexpr int64_t kMaxRows = 1ll << 31;

thread_local char g_err[512] = "";

int fail(int code, const char* fmt, ...) {
  va_list ap;
  va_start(ap, fmt);
  vsnprintf(g_err, sizeof(g_err), fmt, ap);
  va_end(ap);
  return code;
}
#define FA_REQUIRE(cond, ...) \
  do {                         \
    if (!(cond)) return fail(FA_ABI_ERR_INVALID_ARGUMENT, __VA_ARGS__); \
  } while (0)

int done(cudaError_t e, const char* what) {
  if (e != cudaSuccess) return fail(FA_ABI_ERR_CUDA, "%s failed: %s", what, cudaGetErrorString(e));
  return FA_ABI_OK;
}
bool dtype_ok(int dtype) { return dtype == 0 || dtype == 1; }
cudaStream_t st(void* s) { return static_cast<cudaStream_t>(s); }
int sm_count() {
  static int cached[64] = {0};
  int dev = 0, n = 148;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return n;
  if (cached[dev] == 0 && cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) == cudaSuccess) cached[dev] = n;
  return cached[dev] ? cached[dev] : n;
}
// cuTensorMapEncodeTiled, or null if the driver does not have it.
void* tensor_map_encode() {
  static void* fn = [] {
    void* sym = nullptr;
    cudaDriverEntryPointQueryResult qres;
    const cudaError_t e = cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &qres);
    return e == cudaSuccess && qres == cudaDriverEntryPointSuccess ? sym : nullptr;
  }();
  return fn;
}

}  // namespace
