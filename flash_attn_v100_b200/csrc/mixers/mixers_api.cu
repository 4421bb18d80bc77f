// C-ABI entry points of the further sequence mixers (see include/fa_b200_mixers.h): argument checks and launches.
#include "../../../include/fa_b200_mixers.h"

#include "../api_common.cuh"
#include "../hybrid/hybrid_common.cuh"
#include "kv_attention.cuh"
#include "recurrence.cuh"

namespace {

using fa::hybrid::bf16;
namespace mx = fa::mixers;

// Calls fn<T>(args...) for the element type of `dtype`.
#define FAM_DISPATCH(dtype, fn, ...) ((dtype) == FAM_BF16 ? fn<bf16>(__VA_ARGS__) : fn<float>(__VA_ARGS__))

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

int check_recurrence(const FamRecurrence* p, mx::RecurrenceArgs& a) {
  FA_REQUIRE(p != nullptr && dtype_ok(p->dtype), "null arguments or unknown dtype");
  FA_REQUIRE(p->x && p->state && p->slots && p->starts && p->out && p->status, "null pointer");
  FA_REQUIRE(p->heads > 0 && p->heads < 65536 && p->groups > 0 && p->heads % p->groups == 0, "heads=%d are not whole groups of %d", p->heads, p->groups);
  FA_REQUIRE(p->dk > 0 && p->dk <= 1024 && p->dv > 0 && p->dv <= (1 << 20) && p->n_slots > 0, "bad sizes: dk=%d dv=%d slots=%d", p->dk, p->dv, p->n_slots);
  FA_REQUIRE(p->n_seq >= 0 && p->total >= p->n_seq && p->total < kMaxRows && (p->cu_seqlens != nullptr || p->total == p->n_seq),
             "bad sizes: n_seq=%d total=%lld", p->n_seq, (long long)p->total);
  const int64_t kd = (int64_t)p->groups * p->dk, vd = (int64_t)p->heads * p->dv;
  FA_REQUIRE(p->off_q >= 0 && p->off_k >= 0 && p->off_v >= 0 && p->off_q + kd <= p->stride && p->off_k + kd <= p->stride && p->off_v + vd <= p->stride,
             "a column range ends past the row stride");
  a = mx::RecurrenceArgs{};
  a.qkv = p->x; a.stride = p->stride; a.off_q = p->off_q; a.off_k = p->off_k; a.off_v = p->off_v;
  a.heads = p->heads; a.kv_rep = p->heads / p->groups; a.dk = p->dk; a.dv = p->dv; a.q_scale = p->q_scale;
  a.la = p->la; a.b = p->b; a.floor = p->floor; a.n0 = p->n0; a.norm = p->norm; a.norm_eps = p->norm_eps; a.skip = p->skip;
  a.state = p->state; a.n_slots = p->n_slots; a.slots = p->slots; a.starts = p->starts; a.cu = p->cu_seqlens; a.n_seq = p->n_seq; a.total = p->total;
  a.out = p->out; a.status = p->status;
  return FAM_OK;
}

size_t segment_bytes(const mx::RecurrenceArgs& a, int segs) {
  if (segs <= 1) return 0;
  const size_t n = (size_t)a.n_seq * segs * a.heads;
  return n * ((size_t)a.dk * a.dv + a.dk + 4) * sizeof(float);
}

int check_pages(const FamPages* p) {
  FA_REQUIRE(p != nullptr && dtype_ok(p->dtype), "null arguments or unknown dtype");
  FA_REQUIRE(p->k_pool && p->v_pool && p->block_table && p->status, "null pointer");
  FA_REQUIRE(p->n_blocks > 0 && p->max_blocks > 0 && p->n_seq > 0 && p->rows >= 0 && p->rows < kMaxRows, "bad cache sizes");
  FA_REQUIRE(p->kv_heads > 0 && p->heads > 0 && p->heads < 65536 && p->heads % p->kv_heads == 0 && p->dim > 0 && p->vdim > 0 && p->dim <= 8192 && p->vdim <= 8192,
             "bad sizes: heads=%d kv_heads=%d dim=%d vdim=%d", p->heads, p->kv_heads, p->dim, p->vdim);
  return FAM_OK;
}
mx::Paging paging(const FamPages* p) { return {p->n_blocks, p->block_table, p->max_blocks, p->n_seq, p->tok_seq, p->positions}; }

}  // namespace

extern "C" {

const char* fam_last_error(void) { return g_err; }

size_t fam_recurrence_workspace(const FamRecurrence* p) {
  if (p == nullptr || p->dtype != FAM_BF16 || p->cu_seqlens == nullptr || p->n_seq <= 0 || p->groups <= 0 || p->max_len <= 0) return 0;
  mx::RecurrenceArgs a{};
  a.heads = p->heads; a.kv_rep = p->heads / p->groups; a.dk = p->dk; a.dv = p->dv; a.n_seq = p->n_seq;
  if (a.kv_rep <= 0 || a.dk <= 0 || a.dv <= 0) return 0;
  int len = 0;
  return segment_bytes(a, mx::recurrence_segments(a.n_seq, a.heads, a.kv_rep, a.dk, a.dv, p->max_len, sm_count(), &len));
}

int fam_recurrence(const FamRecurrence* p, void* stream) {
  mx::RecurrenceArgs a;
  const int rc = check_recurrence(p, a);
  if (rc != FAM_OK) return rc;
  FA_REQUIRE(p->la && p->b, "null pointer");
  FA_REQUIRE(p->floor == nullptr || (p->n0 != nullptr && p->norm != nullptr), "floor needs n0 and norm");
  if (p->dtype == FAM_BF16 && p->cu_seqlens != nullptr && mx::recurrence_tc5_supported(a)) {
    FA_REQUIRE(p->max_len > 0, "prompts need max_len");
    a.max_segs = mx::recurrence_segments(a.n_seq, a.heads, a.kv_rep, a.dk, a.dv, p->max_len, sm_count(), &a.seg_len);
    const size_t need = segment_bytes(a, a.max_segs);
    FA_REQUIRE((size_t)p->workspace_bytes >= need && (need == 0 || (p->workspace != nullptr && aligned16(p->workspace))),
               "the workspace has %lld bytes, %zu (16-byte aligned) are needed", (long long)p->workspace_bytes, need);
    const size_t n = (size_t)a.n_seq * a.max_segs * a.heads;
    a.seg_state = static_cast<float*>(p->workspace);
    a.seg_norm = need ? a.seg_state + n * a.dk * a.dv : nullptr;
    a.seg_log = need ? a.seg_norm + n * a.dk : nullptr;
    void* enc = tensor_map_encode();
    if (enc == nullptr) return fail(FAM_ERR_CUDA, "cuTensorMapEncodeTiled is not available from the driver");
    return done(mx::launch_recurrence_tc5(a, enc, st(stream)), "recurrence_tc5");
  }
  return done(FAM_DISPATCH(p->dtype, mx::launch_recurrence_scan, a, st(stream)), "recurrence_scan");
}

int fam_max_gates(const void* x, int64_t stride, int off_i, int off_f, int heads, const void* bias_i, const void* bias_f, float cap, float* m,
                  const float* norm, float* n0, int dk, int n_slots, const int32_t* slots, const int32_t* starts, const int32_t* cu_seqlens, int n_seq,
                  int64_t total, float* la, float* b, float* floor, int32_t* status, int dtype, void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(x && bias_i && bias_f && m && norm && n0 && slots && starts && la && b && floor && status, "null pointer");
  FA_REQUIRE(heads > 0 && heads < 65536 && dk > 0 && n_slots > 0 && cap > 0.f, "bad sizes: heads=%d dk=%d cap=%g", heads, dk, (double)cap);
  FA_REQUIRE(n_seq >= 0 && total >= n_seq && total < kMaxRows && (cu_seqlens != nullptr || total == n_seq), "bad sizes: n_seq=%d total=%lld", n_seq, (long long)total);
  FA_REQUIRE(off_i >= 0 && off_f >= 0 && off_i + (int64_t)heads <= stride && off_f + (int64_t)heads <= stride, "a column range ends past the row stride");
  mx::MaxGateArgs a{x, stride, off_i, off_f, heads, bias_i, bias_f, cap, m, norm, n0, dk, n_slots, slots, starts, cu_seqlens, n_seq, total, la, b, floor, status};
  return done(FAM_DISPATCH(dtype, mx::launch_max_gates, a, st(stream)), "max_gates");
}

int fam_step_gates(const void* x, int64_t stride, int off, int heads, const float* bias, const float* a_log, int64_t total, float* la, float* b, int dtype,
                   void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(x && bias && a_log && la && b, "null pointer");
  FA_REQUIRE(heads > 0 && off >= 0 && off + (int64_t)heads <= stride && total >= 0 && total < kMaxRows, "bad sizes: heads=%d off=%d total=%lld", heads, off,
             (long long)total);
  mx::StepGateArgs a{x, stride, off, heads, bias, a_log, total, la, b};
  return done(FAM_DISPATCH(dtype, mx::launch_step_gates, a, st(stream)), "step_gates");
}

int fam_conv_silu(const void* x, int64_t stride, int off, int channels, int taps, const void* w, const void* bias, void* ring, int n_slots,
                  const int32_t* slots, const int32_t* starts, const int32_t* cu_seqlens, const int32_t* tok_seq, const int32_t* positions, int n_seq,
                  int64_t total, void* out, int32_t* status, int dtype, void* stream) {
  FA_REQUIRE(dtype_ok(dtype), "unknown dtype %d", dtype);
  FA_REQUIRE(x && w && bias && ring && slots && starts && tok_seq && positions && out && status, "null pointer");
  FA_REQUIRE(channels > 0 && taps > 0 && taps < 65536 && off >= 0 && off + (int64_t)channels <= stride && n_slots > 0, "bad sizes: channels=%d taps=%d off=%d",
             channels, taps, off);
  FA_REQUIRE(n_seq >= 0 && total >= n_seq && total < kMaxRows && (cu_seqlens != nullptr || total == n_seq), "bad sizes: n_seq=%d total=%lld", n_seq, (long long)total);
  mx::ConvArgs a{x, stride, off, channels, taps, w, bias, ring, n_slots, slots, starts, cu_seqlens, tok_seq, positions, n_seq, total, out, status};
  return done(FAM_DISPATCH(dtype, mx::launch_conv_silu, a, st(stream)), "conv_silu");
}

int fam_recurrence_step_supported(int dk, int dv) {
  mx::RecurrenceArgs a{};
  a.dk = dk; a.dv = dv;
  return mx::recurrence_step_supported(a) ? 1 : 0;
}

int fam_max_gate_step(const FamRecurrence* p, int off_i, int off_f, const void* bias_i, const void* bias_f, float cap, float* m, void* stream) {
  mx::MaxGateStepArgs a{};
  const int rc = check_recurrence(p, a.r);
  if (rc != FAM_OK) return rc;
  FA_REQUIRE(p->norm && bias_i && bias_f && m, "null pointer");
  FA_REQUIRE(cap > 0.f && off_i >= 0 && off_f >= 0 && off_i + (int64_t)p->heads <= p->stride && off_f + (int64_t)p->heads <= p->stride,
             "a column range ends past the row stride");
  if (p->cu_seqlens != nullptr || !mx::recurrence_step_supported(a.r)) return fail(FAM_ERR_UNSUPPORTED, "max_gate_step is not built for dk=%d dv=%d", p->dk, p->dv);
  a.off_i = off_i; a.off_f = off_f; a.bias_i = bias_i; a.bias_f = bias_f; a.cap = cap; a.m = m;
  return done(FAM_DISPATCH(p->dtype, mx::launch_max_gate_step, a, sm_count(), st(stream)), "max_gate_step");
}

int fam_ssd_step(const FamRecurrence* p, int off_dt, const float* dt_bias, const float* a_log, const void* conv_w, const void* conv_b, void* ring, int taps,
                 void* stream) {
  mx::SsdStepArgs a{};
  const int rc = check_recurrence(p, a.r);
  if (rc != FAM_OK) return rc;
  FA_REQUIRE(p->skip && dt_bias && a_log && conv_w && conv_b && ring, "null pointer");
  FA_REQUIRE(taps > 0 && off_dt >= 0 && off_dt + (int64_t)p->heads <= p->stride, "bad sizes: taps=%d off_dt=%d", taps, off_dt);
  FA_REQUIRE(p->off_k == p->off_v + p->heads * p->dv && p->off_q == p->off_k + p->groups * p->dk, "the columns of v, k and q must be adjacent");
  if (p->cu_seqlens != nullptr || !mx::recurrence_step_supported(a.r)) return fail(FAM_ERR_UNSUPPORTED, "ssd_step is not built for dk=%d dv=%d", p->dk, p->dv);
  a.off_dt = off_dt; a.dt_bias = dt_bias; a.a_log = a_log; a.conv_w = conv_w; a.conv_b = conv_b; a.ring = ring; a.taps = taps;
  return done(FAM_DISPATCH(p->dtype, mx::launch_ssd_step, a, sm_count(), st(stream)), "ssd_step");
}

int fam_kv_prep(const FamPages* p, const void* x, int64_t stride, int off_q, int off_k, int off_v, const void* wq, const void* wk, float eps,
                const void* v_first, int64_t first_stride, float lambda, void* q_out, void* k_out, void* v_out, void* stream) {
  const int rc = check_pages(p);
  if (rc != FAM_OK) return rc;
  FA_REQUIRE(x && wq && wk && q_out && p->tok_seq && p->positions, "null pointer");
  FA_REQUIRE(off_q >= 0 && off_k >= 0 && off_v >= 0 && off_q + (int64_t)p->heads * p->dim <= stride && off_k + (int64_t)p->kv_heads * p->dim <= stride &&
                 off_v + (int64_t)p->kv_heads * p->vdim <= stride,
             "a column range ends past the row stride");
  mx::KvPrepArgs a{x, stride, off_q, off_k, off_v, p->heads, p->kv_heads, p->dim, p->vdim, wq, wk, eps, v_first, first_stride, lambda, q_out, k_out, v_out,
                   p->k_pool, p->v_pool, paging(p), p->rows, p->status};
  return done(FAM_DISPATCH(p->dtype, mx::launch_kv_prep, a, st(stream)), "kv_prep");
}

size_t fam_kv_attention_workspace(const FamPages* p, int chunk) {
  if (p == nullptr || p->dtype != FAM_BF16 || p->rows <= 0 || p->heads <= 0 || p->kv_heads <= 0) return 0;
  const int64_t splits = mx::kv_decode_splits(p->rows, p->kv_heads, chunk, p->max_blocks, sm_count());
  return splits > 1 ? (size_t)(p->rows * splits * p->heads * ((int64_t)p->vdim + 2) * 4) : 0;
}

int fam_kv_attention(const FamPages* p, const void* q, const float* slopes, const void* gate, int64_t gate_stride, int chunk, float scale, void* out,
                     int64_t out_stride, void* workspace, size_t workspace_bytes, void* stream) {
  const int rc = check_pages(p);
  if (rc != FAM_OK) return rc;
  const int64_t ov = (int64_t)p->heads * p->vdim;
  FA_REQUIRE(q && out && p->tok_seq && p->positions, "null pointer");
  FA_REQUIRE(chunk >= 0 && out_stride >= ov && (gate == nullptr || gate_stride >= ov), "bad sizes: chunk=%d out_stride=%lld gate_stride=%lld", chunk,
             (long long)out_stride, (long long)gate_stride);
  mx::KvAttentionArgs a{};
  a.q = q; a.k_pool = p->k_pool; a.v_pool = p->v_pool; a.pg = paging(p); a.slopes = slopes; a.gate = gate; a.gate_stride = gate_stride;
  a.heads = p->heads; a.kv_heads = p->kv_heads; a.dim = p->dim; a.vdim = p->vdim; a.chunk = chunk; a.scale = scale; a.out = out; a.out_stride = out_stride;
  a.rows = p->rows; a.status = p->status;
  if (p->dtype == FAM_BF16 && mx::kv_decode_supported(a)) {
    const size_t need = fam_kv_attention_workspace(p, chunk);
    FA_REQUIRE(workspace_bytes >= need && (need == 0 || (workspace != nullptr && aligned16(workspace))),
               "the workspace has %zu bytes, %zu (16-byte aligned) are needed", workspace_bytes, need);
    a.splits = mx::kv_decode_splits(p->rows, p->kv_heads, chunk, p->max_blocks, sm_count());
    a.part_o = static_cast<float*>(workspace);
    a.part_ml = need ? a.part_o + p->rows * a.splits * p->heads * p->vdim : nullptr;
    return done(mx::launch_kv_decode(a, st(stream)), "kv_decode");
  }
  return done(FAM_DISPATCH(p->dtype, mx::launch_kv_attention, a, st(stream)), "kv_attention");
}

int fam_kv_gather(const FamPages* p, const int32_t* piece_seq, const int32_t* piece_key0, const int32_t* cu_kv, int pieces, int64_t total_kv, void* k, void* v,
                  void* stream) {
  const int rc = check_pages(p);
  if (rc != FAM_OK) return rc;
  FA_REQUIRE(piece_seq && piece_key0 && cu_kv && k && v, "null pointer");
  FA_REQUIRE(pieces > 0 && total_kv >= 0 && total_kv < kMaxRows, "bad sizes: pieces=%d total_kv=%lld", pieces, (long long)total_kv);
  mx::KvGatherArgs a{p->k_pool, p->v_pool, p->n_blocks, p->block_table, p->max_blocks, p->n_seq, piece_seq, piece_key0, cu_kv, pieces, total_kv,
                     p->kv_heads, p->dim, p->vdim, k, v, p->status};
  return done(FAM_DISPATCH(p->dtype, mx::launch_kv_gather, a, st(stream)), "kv_gather");
}

int fam_kv_prefill_supported(int heads, int kv_heads, int dim, int vdim, float scale, int dtype) {
  return dtype == FAM_BF16 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && mx::kv_prefill_supported(heads, kv_heads, dim, vdim, scale) ? 1 : 0;
}

int fam_kv_prefill(const void* q, const void* k, const void* v, const int32_t* cu_q, const int32_t* cu_kv, int pieces, int max_q, int64_t total_q,
                   int64_t total_kv, int heads, int kv_heads, int dim, int vdim, float scale, const float* slopes, const void* gate,
                   int64_t gate_stride, void* out, int64_t out_stride, int32_t* status, void* stream) {
  FA_REQUIRE(q && k && v && cu_q && cu_kv && slopes && out && status, "null pointer");
  if (!fam_kv_prefill_supported(heads, kv_heads, dim, vdim, scale, FAM_BF16))
    return fail(FAM_ERR_UNSUPPORTED, "kv_prefill is not built for heads=%d/%d dim=%d vdim=%d scale=%g", heads, kv_heads, dim, vdim, (double)scale);
  const int64_t ov = (int64_t)heads * vdim;
  FA_REQUIRE(pieces > 0 && max_q > 0 && total_q >= 0 && total_q < kMaxRows && total_kv >= total_q && total_kv < kMaxRows, "bad sizes: pieces=%d max_q=%d", pieces,
             max_q);
  FA_REQUIRE(aligned16(q) && aligned16(k) && aligned16(v) && aligned16(out) && out_stride % 8 == 0 && out_stride >= ov,
             "q, k, v and out must be 16-byte aligned, out_stride a multiple of 8");
  FA_REQUIRE(gate == nullptr || (aligned16(gate) && gate_stride % 8 == 0 && gate_stride >= ov), "gate must be 16-byte aligned, gate_stride a multiple of 8");
  void* enc = tensor_map_encode();
  if (enc == nullptr) return fail(FAM_ERR_CUDA, "cuTensorMapEncodeTiled is not available from the driver");
  mx::KvPrefillArgs a{q, k, v, cu_q, cu_kv, pieces, max_q, total_q, total_kv, heads, kv_heads, dim, vdim, scale, slopes, gate, gate_stride, out, out_stride, status};
  return done(mx::launch_kv_prefill(a, enc, st(stream)), "kv_prefill");
}

}  // extern "C"
