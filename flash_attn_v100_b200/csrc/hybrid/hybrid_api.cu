// C-ABI entry points of the hybrid decoder's operators (see include/fa_b200_hybrid.h): argument checks and launches.
#include "../../../include/fa_b200_hybrid.h"

#include "../api_common.cuh"
#include "hybrid_common.cuh"
#include "latent_attention.cuh"
#include "latent_prefill.cuh"
#include "latent_prep.cuh"
#include "lightning.cuh"

namespace {

using fa::hybrid::bf16;

// Calls fn<T>(args...) for the element type of `dtype`.
#define FAH_DISPATCH(dtype, fn, ...) ((dtype) == FAH_BF16 ? fn<bf16>(__VA_ARGS__) : fn<float>(__VA_ARGS__))

}  // namespace

extern "C" {

const char* fah_last_error(void) { return g_err; }

size_t fah_lightning_workspace(int n_seq, int heads, int dk, int dv, int max_len, int dtype) {
  if (dtype != FAH_BF16 || n_seq <= 0 || heads <= 0 || dk <= 0 || dv <= 0 || max_len <= 0) return 0;
  int seg_len = 0;
  const int segs = fa::hybrid::lightning_segments(n_seq, heads, dk, dv, max_len, sm_count(), &seg_len);
  return segs > 1 ? (size_t)n_seq * segs * heads * dk * dv * sizeof(float) : 0;
}

int fah_lightning(const void* qkv, int64_t stride, int off_q, int off_k, int off_v, int heads, int dk, int dv, const float* decay, float* state,
                  int n_slots, const int32_t* slots, const int32_t* starts, const int32_t* cu_seqlens, int n_seq, int max_len, int64_t tokens,
                  void* out, void* workspace, size_t workspace_bytes, int32_t* status, int dtype, void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(qkv && decay && state && slots && starts && out && status, "null pointer");
  FA_REQUIRE(heads > 0 && heads < 65536 && dk > 0 && dv > 0 && n_slots > 0, "bad sizes: heads=%d dk=%d dv=%d slots=%d", heads, dk, dv, n_slots);
  FA_REQUIRE(dk <= 1536, "dk=%d is larger than the 1536 the kernels are built for", dk);
  FA_REQUIRE(n_seq >= 0 && tokens >= n_seq && tokens < kMaxRows && (cu_seqlens != nullptr || tokens == n_seq), "bad sizes: n_seq=%d tokens=%lld", n_seq,
              (long long)tokens);
  FA_REQUIRE(off_q >= 0 && off_k >= 0 && off_v >= 0 && off_q + (int64_t)heads * dk <= stride && off_k + (int64_t)heads * dk <= stride &&
                  off_v + (int64_t)heads * dv <= stride,
              "a column range ends past the row stride");
  fa::hybrid::LightningArgs a{};
  a.qkv = qkv; a.stride = stride; a.off_q = off_q; a.off_k = off_k; a.off_v = off_v;
  a.heads = heads; a.dk = dk; a.dv = dv; a.decay = decay; a.state = state; a.n_slots = n_slots; a.slots = slots; a.starts = starts;
  a.cu = cu_seqlens; a.n_seq = n_seq; a.total = tokens; a.out = out; a.status = status;
  if (fa::hybrid::lightning_decode_supported(a))
    return done(FAH_DISPATCH(dtype, fa::hybrid::launch_lightning_decode, a, sm_count(), st(stream)), "lightning_decode");
  if (dtype == FAH_BF16 && fa::hybrid::lightning_chunk_supported(a)) {
    FA_REQUIRE(max_len > 0, "prompts need max_len");
    const size_t need = fah_lightning_workspace(n_seq, heads, dk, dv, max_len, dtype);
    FA_REQUIRE(workspace_bytes >= need && (need == 0 || (workspace != nullptr && (reinterpret_cast<uintptr_t>(workspace) & 15) == 0)),
                "the workspace has %zu bytes, %zu (16-byte aligned) are needed", workspace_bytes, need);
    a.max_segs = fa::hybrid::lightning_segments(n_seq, heads, dk, dv, max_len, sm_count(), &a.seg_len);
    a.seg_state = static_cast<float*>(workspace);
    return done(fa::hybrid::launch_lightning_chunk(a, st(stream)), "lightning_chunk");
  }
  return done(FAH_DISPATCH(dtype, fa::hybrid::launch_lightning_scan, a, st(stream)), "lightning_scan");
}

int fah_latent_prep(const void* down, int64_t down_stride, int off_q, int q_rank, int off_kv, int kv_rank, int off_r, int rot_dim, const void* wq,
                    const void* wkv, float eps, const float* cos_t, const float* sin_t, void* cq, void* c_out, void* r_out, void* pool,
                    int pool_stride, int n_blocks, const int32_t* block_table, int max_blocks, int n_seq, const int32_t* tok_seq,
                    const int32_t* positions, int64_t rows, int32_t* status, int dtype, void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(down && wq && wkv && cos_t && sin_t && cq && pool && block_table && tok_seq && positions && status, "null pointer");
  FA_REQUIRE(q_rank > 0 && kv_rank > 0 && rot_dim > 0 && rot_dim % 2 == 0, "bad sizes: q_rank=%d kv_rank=%d rot_dim=%d", q_rank, kv_rank, rot_dim);
  FA_REQUIRE(off_q >= 0 && off_kv >= 0 && off_r >= 0 && off_q + (int64_t)q_rank <= down_stride && off_kv + (int64_t)kv_rank <= down_stride &&
                  off_r + (int64_t)rot_dim <= down_stride,
              "a column range ends past the row stride");
  FA_REQUIRE(pool_stride >= kv_rank + rot_dim && n_blocks > 0 && max_blocks > 0 && n_seq > 0 && rows >= 0 && rows < kMaxRows, "bad cache sizes");
  fa::hybrid::LatentPrepArgs a{down, down_stride, off_q, q_rank, off_kv, kv_rank, off_r, rot_dim, wq, wkv, eps, cos_t, sin_t, cq, c_out, r_out, pool,
                               pool_stride, n_blocks, block_table, max_blocks, n_seq, tok_seq, positions, rows, status};
  return done(FAH_DISPATCH(dtype, fa::hybrid::launch_latent_prep, a, st(stream)), "latent_prep");
}

int fah_rotate_heads(void* q, const float* cos_t, const float* sin_t, int64_t rows, int heads, int head_stride, int off, int rot_dim, int dtype,
                     void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(q && cos_t && sin_t, "null pointer");
  FA_REQUIRE(rows >= 0 && rows < kMaxRows && heads > 0 && off >= 0 && rot_dim >= 0 && rot_dim % 2 == 0 && off + rot_dim <= head_stride,
              "bad sizes: heads=%d off=%d rot_dim=%d head_stride=%d", heads, off, rot_dim, head_stride);
  return done(FAH_DISPATCH(dtype, fa::hybrid::launch_rotate_heads, q, cos_t, sin_t, rows, heads, head_stride, off, rot_dim, st(stream)), "rotate_heads");
}

size_t fah_latent_attention_workspace(int heads, int kv_rank, int rot_dim, int64_t rows, int dtype) {
  if (dtype != FAH_BF16 || heads <= 0 || rows <= 0 || kv_rank <= 0) return 0;
  const int64_t n = fa::hybrid::latent_decode_ctas(heads, sm_count());
  return (size_t)(n * 2 * heads * ((int64_t)kv_rank + 2) * 4 + (rows + 1) * 4);
}

int fah_latent_attention(const void* q_abs, const void* q, int q_stride, int q_off, const float* cos_t, const float* sin_t, const void* pool,
                         int pool_stride, int n_blocks, const int32_t* block_table, int max_blocks, int n_seq, const int32_t* tok_seq,
                         const int32_t* positions, const void* gate, int64_t gate_stride, int heads, int kv_rank, int rot_dim, float scale, void* out,
                         int64_t rows, void* workspace, size_t workspace_bytes, int32_t* status, int dtype, void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(q_abs && q && cos_t && sin_t && pool && block_table && tok_seq && positions && out && status, "null pointer");
  FA_REQUIRE(heads > 0 && heads < 65536 && kv_rank > 0 && kv_rank <= 16384 && rot_dim >= 0 && rot_dim % 2 == 0 && q_off >= 0 && q_off + rot_dim <= q_stride,
              "bad sizes: heads=%d kv_rank=%d rot_dim=%d", heads, kv_rank, rot_dim);
  FA_REQUIRE(pool_stride >= kv_rank + rot_dim && n_blocks > 0 && max_blocks > 0 && n_seq > 0 && rows >= 0 && rows < kMaxRows, "bad cache sizes");
  FA_REQUIRE(gate == nullptr || gate_stride >= heads, "gate_stride=%lld is smaller than heads=%d", (long long)gate_stride, heads);
  fa::hybrid::LatentAttentionArgs a{};
  a.q_abs = q_abs; a.q = q; a.q_stride = q_stride; a.q_off = q_off; a.cos_t = cos_t; a.sin_t = sin_t; a.pool = pool; a.pool_stride = pool_stride;
  a.n_blocks = n_blocks; a.block_table = block_table; a.max_blocks = max_blocks; a.n_seq = n_seq; a.tok_seq = tok_seq; a.positions = positions;
  a.gate = gate; a.gate_stride = gate_stride; a.heads = heads; a.kv_rank = kv_rank; a.rot_dim = rot_dim; a.scale = scale; a.out = out; a.rows = rows;
  a.status = status;
  if (dtype == FAH_BF16 && fa::hybrid::latent_decode_supported(a)) {
    const size_t need = fah_latent_attention_workspace(heads, kv_rank, rot_dim, rows, dtype);
    FA_REQUIRE(workspace_bytes >= need && (need == 0 || (workspace != nullptr && (reinterpret_cast<uintptr_t>(workspace) & 15) == 0)),
                "the workspace has %zu bytes, %zu (16-byte aligned) are needed", workspace_bytes, need);
    a.n_cta = fa::hybrid::latent_decode_ctas(heads, sm_count());
    a.part_o = static_cast<float*>(workspace);
    a.part_ml = a.part_o + (int64_t)a.n_cta * 2 * heads * kv_rank;
    a.row_tiles = reinterpret_cast<int32_t*>(a.part_ml + (int64_t)a.n_cta * 2 * heads * 2);
    void* enc = tensor_map_encode();
    if (enc == nullptr) return fail(FAH_ERR_CUDA, "cuTensorMapEncodeTiled is not available from the driver");
    return done(fa::hybrid::launch_latent_decode(a, enc, st(stream)), "latent_decode");
  }
  return done(FAH_DISPATCH(dtype, fa::hybrid::launch_latent_attention, a, st(stream)), "latent_attention");
}

int fah_latent_prefill_supported(int dim, int rot_dim, int vdim, float scale, int dtype) {
  return dtype == FAH_BF16 && fa::hybrid::latent_prefill_supported(dim, rot_dim, vdim, scale) ? 1 : 0;
}

int fah_latent_prefill(const void* q, const void* kv, const void* kr, const void* gate, int64_t gate_stride, const int32_t* cu_q,
                       const int32_t* cu_kv, int n_seq, int max_q, int64_t total_q, int64_t total_kv, int heads, int dim, int rot_dim, int vdim,
                       float scale, void* out, int32_t* status, void* stream) {
  FA_REQUIRE(q && kv && kr && cu_q && cu_kv && out && status, "null pointer");
  if (!fa::hybrid::latent_prefill_supported(dim, rot_dim, vdim, scale))
    return fail(FAH_ERR_UNSUPPORTED, "latent_prefill is not built for dim=%d rot_dim=%d vdim=%d scale=%g", dim, rot_dim, vdim, (double)scale);
  FA_REQUIRE(heads > 0 && n_seq > 0 && max_q > 0 && total_q >= 0 && total_q < kMaxRows && total_kv >= total_q && total_kv < kMaxRows,
              "bad sizes: heads=%d n_seq=%d max_q=%d total_q=%lld total_kv=%lld", heads, n_seq, max_q, (long long)total_q, (long long)total_kv);
  FA_REQUIRE(gate == nullptr || gate_stride >= heads, "gate_stride=%lld is smaller than heads=%d", (long long)gate_stride, heads);
  for (const void* p : {q, kv, kr, (const void*)out})
    FA_REQUIRE((reinterpret_cast<uintptr_t>(p) & 15) == 0, "q, kv, kr and out must be 16-byte aligned");
  void* enc = tensor_map_encode();
  if (enc == nullptr) return fail(FAH_ERR_CUDA, "cuTensorMapEncodeTiled is not available from the driver");
  fa::hybrid::LatentPrefillArgs a{q, kv, kr, gate, gate_stride, cu_q, cu_kv, n_seq, max_q, total_q, total_kv, heads, dim, rot_dim, vdim, scale, out,
                                  status};
  return done(fa::hybrid::launch_latent_prefill(a, enc, st(stream)), "latent_prefill");
}

int fah_latent_gather(const void* pool, int pool_stride, int n_blocks, const int32_t* block_table, int max_blocks, int n_seq, const int32_t* cu_kv,
                      int64_t total_kv, int kv_rank, int rot_dim, void* c, void* r, int32_t* status, int dtype, void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(pool && block_table && cu_kv && c && r && status, "null pointer");
  FA_REQUIRE(kv_rank > 0 && rot_dim > 0 && pool_stride >= kv_rank + rot_dim && n_blocks > 0 && max_blocks > 0 && n_seq > 0 && total_kv >= 0 &&
                  total_kv < kMaxRows,
              "bad sizes: kv_rank=%d rot_dim=%d n_seq=%d total_kv=%lld", kv_rank, rot_dim, n_seq, (long long)total_kv);
  fa::hybrid::LatentGatherArgs a{pool, pool_stride, n_blocks, block_table, max_blocks, n_seq, cu_kv, total_kv, kv_rank, rot_dim, c, r, status};
  return done(FAH_DISPATCH(dtype, fa::hybrid::launch_latent_gather, a, st(stream)), "latent_gather");
}

}  // extern "C"
