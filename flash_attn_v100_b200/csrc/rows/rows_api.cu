// C-ABI entry points of the row-wise operators (see include/fa_b200_rows.h): argument checks and launches.
#include "../../../include/fa_b200_rows.h"

#include "../api_common.cuh"
#include "../hybrid/hybrid_common.cuh"
#include "row_ops.cuh"

namespace {

using fa::hybrid::bf16;

// Calls fn<T>(args...) for the element type of `dtype`.
#define FAR_DISPATCH(dtype, fn, ...) ((dtype) == FAR_BF16 ? fn<bf16>(__VA_ARGS__) : fn<float>(__VA_ARGS__))

}  // namespace

extern "C" {

const char* far_last_error(void) { return g_err; }

int far_residual_norm(const FarResidualNorm* n, void* stream) {
  FA_REQUIRE(n != nullptr, "null pointer");
  FA_REQUIRE(dtype_ok(n->dtype), "unknown dtype %d", n->dtype);
  FA_REQUIRE(n->x != nullptr, "x is null");
  FA_REQUIRE(n->rows >= 0 && n->rows < kMaxRows && n->cols > 0, "bad sizes: rows=%lld cols=%d", (long long)n->rows, n->cols);
  FA_REQUIRE(n->embed_mode >= 0 && n->embed_mode <= 2, "embed_mode must be 0, 1 or 2");
  FA_REQUIRE(n->embed_mode == 0 || (n->embed != nullptr && n->tokens != nullptr && n->vocab > 0), "embed_mode %d needs embed, tokens and vocab",
             n->embed_mode);
  FA_REQUIRE(n->delta_w == nullptr || n->delta != nullptr, "delta_w without delta");
  FA_REQUIRE(n->w == nullptr || n->out != nullptr, "w without out");
  FA_REQUIRE((n->w2 == nullptr) == (n->out2 == nullptr) && (n->w2 == nullptr || n->w != nullptr), "w2 and out2 go together, beside w and out");
  for (int k = 0; k < 2; ++k)
    FA_REQUIRE(n->more[k] == nullptr || (n->embed_mode == 2 && n->more_rows[k] != nullptr && n->more_n[k] > 0),
               "a further table needs embed_mode 2, its rows and their number");
  FA_REQUIRE(n->embed_scale == 1.f || n->embed_mode == 2, "embed_scale needs embed_mode 2");
  fa::hybrid::ResidualNormArgs a{n->x, n->delta, n->delta_w, n->embed, n->tokens, n->embed_mode, n->w, n->out, n->rows, n->cols, n->vocab, n->eps,
                                 n->w2, n->out2, n->embed_scale, {n->more[0], n->more[1]}, {n->more_rows[0], n->more_rows[1]},
                                 {n->more_n[0], n->more_n[1]}};
  return done(FAR_DISPATCH(n->dtype, fa::hybrid::launch_residual_norm, a, st(stream)), "residual_norm");
}

int far_gated_norm(const void* o, const void* g, int64_t g_stride, const void* w, void* out, int64_t out_stride, int64_t rows, int cols, int group,
                   int silu_first, float eps, int dtype, void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(o && g && w && out, "null pointer");
  FA_REQUIRE(rows >= 0 && rows < kMaxRows && cols > 0 && g_stride >= cols && out_stride >= cols, "bad sizes: rows=%lld cols=%d", (long long)rows, cols);
  FA_REQUIRE(group > 0 && cols % group == 0 && cols / group < 65536, "cols=%d are not whole groups of %d", cols, group);
  fa::hybrid::GatedNormArgs a{o, g, g_stride, w, out, out_stride, rows, cols, group, eps, silu_first};
  return done(FAR_DISPATCH(dtype, fa::hybrid::launch_gated_norm, a, st(stream)), "gated_norm");
}

int far_gelu(const void* z, int64_t z_stride, void* out, int64_t out_stride, int64_t rows, int n, int dtype, void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(z && out, "null pointer");
  FA_REQUIRE(rows >= 0 && rows < kMaxRows && n > 0 && z_stride >= n && out_stride >= n, "bad sizes: rows=%lld n=%d", (long long)rows, n);
  return done(FAR_DISPATCH(dtype, fa::hybrid::launch_gelu, z, z_stride, out, out_stride, rows, n, st(stream)), "gelu");
}

int far_bigram_rows(const int64_t* tokens, const int32_t* cu_seqlens, const int32_t* starts, const int32_t* slots, int32_t* last, int n_slots, int n_seq,
                    int64_t total, int64_t buckets, int64_t mul_prev, int64_t mul_cur, int32_t* out, int32_t* status, void* stream) {
  FA_REQUIRE(tokens && starts && slots && last && out && status, "null pointer");
  FA_REQUIRE(n_slots > 0 && n_seq >= 0 && total >= n_seq && total < kMaxRows && (cu_seqlens != nullptr || total == n_seq), "bad sizes: n_seq=%d total=%lld",
             n_seq, (long long)total);
  FA_REQUIRE(buckets > 0 && buckets < kMaxRows - 1 && mul_prev >= 0 && mul_cur >= 0 && mul_prev < kMaxRows && mul_cur < kMaxRows,
             "bad constants: buckets=%lld mul_prev=%lld mul_cur=%lld", (long long)buckets, (long long)mul_prev, (long long)mul_cur);
  return done(fa::hybrid::launch_bigram_rows(tokens, cu_seqlens, starts, slots, last, n_slots, n_seq, total, buckets, mul_prev, mul_cur, out, status,
                                             st(stream)),
              "bigram_rows");
}

int far_clamped_glu(const void* gu, void* out, int64_t rows, int n, float limit, float alpha, float shift, int dtype, void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(gu && out, "null pointer");
  FA_REQUIRE(rows >= 0 && rows < kMaxRows && n > 0, "bad sizes: rows=%lld n=%d", (long long)rows, n);
  return done(FAR_DISPATCH(dtype, fa::hybrid::launch_clamped_glu, gu, out, rows, n, limit, alpha, shift, st(stream)), "clamped_glu");
}

int far_side_gate(const void* z, const void* side, const int64_t* tokens, int vocab, int64_t side_stride, int off, void* out, int64_t rows,
                  int n, int dtype, void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(z && side && tokens && out, "null pointer");
  FA_REQUIRE(rows >= 0 && rows < kMaxRows && n > 0 && vocab > 0 && off >= 0 && off + (int64_t)n <= side_stride, "bad sizes: rows=%lld n=%d off=%d",
              (long long)rows, n, off);
  return done(FAR_DISPATCH(dtype, fa::hybrid::launch_side_gate, z, side, tokens, vocab, side_stride, off, out, rows, n, st(stream)), "side_gate");
}

}  // extern "C"
