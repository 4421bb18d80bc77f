// Gated linear recurrences over prompts on the 5th-generation tensor cores (tcgen05 + TMEM), sm_100a: heads of up to 128 key
// columns and any number of value columns, bfloat16 activations.
//
// In chunks of C = 128 tokens, with L the running sum of la inside the chunk and S the state before it:
//     A  = Q K^T                           O1 = Q S                  S enters as two bfloat16 parts (high, low: about 17 bits)
//     P_ij = A_ij e^(L_i - L_j) b_j, j <= i, as two bfloat16 parts    O2 = P V           P is read from tensor memory
//     o_i = e^(L_i) O1_i + O2_i            dS = K^T V'               v'_j = e^(L_C - L_j) b_j v_j, two bfloat16 parts
//     S  <- e^(L_C) S + dS                 S stays in the threads' registers, fp32
// Decays and weights act on rows of V' and P and on columns of S only, never on Q and K: the 128 value columns of a CTA can
// belong to two heads with the same queries and keys (NH = 2, heads of up to 64 value columns), which share A.
// The normaliser (NORM): n stays in shared memory, fp32; n_i . q_i = e^(L_i) (n . q_i) + sum_j P_ij from the P in registers.
//
// CTA = (segment of a sequence, head or pair of heads, 128 value columns), sixteen warps, all of them with the same role: a warp
// owns 32 lanes (rows) x 32 columns of whatever is in tensor memory; warp 0 issues the MMAs.  Segments let few long sequences
// fill the GPU: a first launch computes what every segment adds to the state, a scan over the segments turns that into the state
// at the start of each, and the main launch then runs all segments side by side.
//
// Tensor memory, 512 columns: A / P of the first head [0, 128)  O1 [128, 256)  O2 [256, 384)  P of the second head / dS [384, 512).
// Shared memory: six tiles of 128 x 128 bfloat16, each two 128-byte-swizzled slabs of 64 columns: Q, K twice, V, and S high and low,
// whose place V' takes once O1 is done.  Q, K and V come by TMA (the next K while this chunk is computed, the next Q once O1 is done,
// the next V once the output, which takes V's place, has been stored, also by TMA).  Rows past a sequence's end have the weight 0.
// Waits are bounded: one that runs out sets the status word and the CTA leaves after another bounded wait for its MMAs and copies.
#include "../hybrid/hybrid_common.cuh"
#include "../tc5.cuh"
#include "../tma3.cuh"
#include "recurrence.cuh"

namespace fa {
namespace mixers {

using hybrid::bf16;

namespace {

constexpr int C = 128;         // tokens per chunk
constexpr int N = 128;         // key and value columns per CTA (padded with zeros)
constexpr int kThreads = 512;
constexpr int SLAB = 128 * 128;
constexpr int TILE = 2 * SLAB;
constexpr float kLog2e = 1.4426950408889634f;

struct Small {                 // behind the tiles
  float2 lb[2][2][C];          // [buffer][head]: running log2 decay and weight of every token
  float wk[2][2][C];           // weight of every token in the state after the chunk
  float dec[2][2];             // log2 decay over the chunk
  float n[N];                  // normaliser
  float n_add[kThreads / 32][N];
  float den[4][C];             // partial n . q of every row, by column group
  uint64_t bars[8];
  uint32_t tmem_slot;
};
constexpr int kTiles = 6;
constexpr int kSmem = 1024 + kTiles * TILE + (int)sizeof(Small);
static_assert(kSmem <= 227 * 1024, "shared memory plan exceeds the SM");

// Byte offset of 16-byte unit `u` (0..15) of row `row` in a tile.
__device__ __forceinline__ uint32_t tile_off(int row, int u) {
  return (uint32_t)((u >> 3) * SLAB + row * 128 + ((u ^ row) & 7) * 16);
}
__device__ __forceinline__ void st_shared(uint32_t addr, const uint4& v) {
  asm volatile("st.shared.v4.b32 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(v.x), "r"(v.y), "r"(v.z), "r"(v.w) : "memory");
}
__device__ __forceinline__ uint4 ld_shared(uint32_t addr) {
  uint4 v;
  asm volatile("ld.shared.v4.b32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ float2 unpack2(uint32_t v) {
  return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u));
}
// Two fp32 numbers as packed (high, low) bfloat16 parts.
__device__ __forceinline__ void split2(float2 v, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf162(v.x, v.y);
  const float2 r = ffma2(unpack2(hi), make_float2(-1.f, -1.f), v);
  lo = pack_bf162(r.x, r.y);
}

template <bool STATE_ONLY, int NH, bool NORM>
__global__ void __launch_bounds__(kThreads, 1)
recurrence_tc5_kernel(const __grid_constant__ CUtensorMap qmap, const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap vmap,
                      const __grid_constant__ CUtensorMap omap, const RecurrenceArgs a) {
  static_assert(NH == 1 || !NORM, "a pair of heads has no normaliser");
  // instruction descriptors: fp32 accumulators, bfloat16 operands, M = 128, N at bit 17; bit 15: A MN-major, bit 16: B MN-major
  constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(128 >> 4) << 24);
  constexpr uint32_t N128 = (uint32_t)(N >> 3) << 17, NPV = (uint32_t)((N / NH) >> 3) << 17;
  constexpr uint32_t IDESC_QK = IDESC | N128, IDESC_B = IDESC | N128 | (1u << 16), IDESC_PV = IDESC | NPV | (1u << 16),
                     IDESC_AB = IDESC | N128 | (1u << 15) | (1u << 16);
  extern __shared__ uint8_t smem_dyn[];
  const uint32_t raw_base = smem_u32(smem_dyn);
  uint8_t* smem = smem_dyn + ((1024u - (raw_base & 1023u)) & 1023u);
  const uint32_t sQ = smem_u32(smem), sK0 = sQ + TILE, sV = sK0 + 2 * TILE, sSh = sV + TILE, sSl = sSh + TILE;
  Small& sm = *reinterpret_cast<Small*>(smem + kTiles * TILE);
  auto bar = [&](int i) { return smem_u32(&sm.bars[i]); };
  const uint32_t bar_a = bar(0), bar_1 = bar(1), bar_o = bar(2), bar_s = bar(3), full_q = bar(4), full_v = bar(5), full_k = bar(6);   // full_k: two

  const int seq = blockIdx.x / a.max_segs, seg = blockIdx.x - seq * a.max_segs;
  const int head0 = blockIdx.y * NH, c0 = blockIdx.z * N, grp = head0 / a.kv_rep;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  long long t0 = a.cu[seq], t1 = a.cu[seq + 1];
  if (t0 < 0) t0 = 0;
  if (t1 > a.total) t1 = a.total;
  const long long seq_end = t1;
  const int seq_len = (int)(t1 - t0);
  t0 += (long long)seg * a.seg_len;
  if (t0 >= t1) return;
  if (t1 > t0 + a.seg_len) t1 = t0 + a.seg_len;
  const bool last_seg = t1 == seq_end;
  if (STATE_ONLY && last_seg) return;              // nothing follows it
  const int n_tok = (int)(t1 - t0), n_chunk = (n_tok + C - 1) / C;

  const int slot = a.slots[seq];
  const bool slot_ok = slot >= 0 && slot < a.n_slots;
  if (!slot_ok && tid == 0) atomicOr(a.status, kStatusBadPageId);
  const long long hs = (long long)a.dk * a.dv;
  const bool segmented = a.max_segs > 1;
  const long long seg_at = ((long long)seq * a.max_segs + seg) * a.heads;      // + head

  // ---- copies: one thread issues them all ------------------------------------------------------------
  const bool copier = tid == kThreads - 32;
  const bool wide_k = a.dk > 64, wide_v = NH == 2 || a.dv - c0 > 64;           // the tile's second slab has columns
  auto load_tile = [&](const CUtensorMap* map, uint32_t dst, uint32_t full, bool wide, int col, int head, int col2, int head2, long long t) {
    mbar_expect_tx(full, wide ? TILE : SLAB);
    tma_load_3d(dst, map, col, head, (int)t, full);
    if (wide) tma_load_3d(dst + SLAB, map, col2, head2, (int)t, full);
  };
  auto load_q = [&](int chunk) { load_tile(&qmap, sQ, full_q, wide_k, 0, grp, 64, grp, t0 + (long long)chunk * C); };
  auto load_k = [&](int chunk) {
    load_tile(&kmap, sK0 + (chunk & 1) * TILE, full_k + (chunk & 1) * 8, wide_k, 0, grp, 64, grp, t0 + (long long)chunk * C);
  };
  auto load_v = [&](int chunk) {
    if (NH == 2) load_tile(&vmap, sV, full_v, true, 0, head0, 0, head0 + 1, t0 + (long long)chunk * C);
    else load_tile(&vmap, sV, full_v, wide_v, c0, head0, c0 + 64, head0, t0 + (long long)chunk * C);
  };
  int n_q = 0, n_k = 0, n_v = 0;                   // (copier) loads issued
  if (copier) {
    for (int i = 0; i < 8; ++i) mbar_init(bar(i), 1);
    mbar_fence_init();
    fence_proxy_async();
    if (!STATE_ONLY) { load_q(0); ++n_q; }
    load_k(0); ++n_k;
    load_v(0); ++n_v;
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm.tmem_slot)), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }

  // ---- decays: warp h < NH turns the chunk's la and b of head h into sums, four tokens per lane -----
  float gl[4], gb[4];
  auto fetch_gates = [&](int chunk) {
    const long long tb = t0 + (long long)chunk * C + lane * 4, at = (long long)(head0 + warp) * a.total + tb;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const bool in = tb + i < t1;
      gl[i] = in ? a.la[at + i] : 0.f;
      gb[i] = in ? a.b[at + i] : 0.f;
    }
  };
  auto put_gates = [&](int buf) {
#pragma unroll
    for (int i = 0; i < 4; ++i) gl[i] *= kLog2e;
    float up = gl[0] + gl[1] + gl[2] + gl[3], down = up;       // sums up to my last token, and from my first token on
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float u = __shfl_up_sync(0xffffffffu, up, o), d = __shfl_down_sync(0xffffffffu, down, o);
      if (lane >= o) up += u;
      if (lane + o < 32) down += d;
    }
    if (lane == 31) sm.dec[buf][warp] = up;
    float before = __shfl_up_sync(0xffffffffu, up, 1), after = __shfl_down_sync(0xffffffffu, down, 1);
    if (lane == 0) before = 0.f;
    if (lane == 31) after = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      before += gl[i];
      sm.lb[buf][warp][lane * 4 + i] = make_float2(before, gb[i]);
    }
#pragma unroll
    for (int i = 3; i >= 0; --i) {                              // (summed from the end: the tokens that matter have small sums)
      sm.wk[buf][warp][lane * 4 + i] = fast_exp2(after) * gb[i];
      after += gl[i];
    }
  };
  if (warp < NH) {
    fetch_gates(0);
    put_gates(0);
  }
  if (NORM && tid < N) {
    float v = 0.f;
    if (!STATE_ONLY && tid < a.dk)
      v = segmented ? a.seg_norm[(seg_at + head0) * a.dk + tid] : a.n0[((long long)seq * a.heads + head0) * a.dk + tid];
    sm.n[tid] = v;
  }
  if (!wide_k || !wide_v) {                                    // slabs that no copy fills
    const uint4 z = make_uint4(0, 0, 0, 0);
    for (int i = tid; i < SLAB / 16; i += kThreads) {
      if (!wide_k) {
        st_shared(sQ + SLAB + i * 16, z);
        st_shared(sK0 + SLAB + i * 16, z);
        st_shared(sK0 + TILE + SLAB + i * 16, z);
      }
      if (!wide_v) st_shared(sV + SLAB + i * 16, z);
    }
    fence_proxy_async();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm.tmem_slot;

  // my place in tensor memory: lane (row) and 32 columns
  const int row = (warp & 3) * 32 + lane, cg = warp >> 2;
  const uint32_t tl = tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)cg * 32u;
  const uint32_t tA = tl, tO1 = tl + 128u, tO2 = tl + 256u, tS = tl + 384u;
  const uint32_t tP = tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)cg * 16u;     // high part; low part 64 columns on
  // ... and what the columns are: a head and its columns from mc on
  const int mh = NH == 2 ? cg >> 1 : 0, mc = NH == 2 ? (cg & 1) * 32 : c0 + cg * 32;

  // ---- state: row `row`, my columns ----------------------------------------------------------------
  float* cache = slot_ok ? a.state + ((long long)slot * a.heads + head0 + mh) * hs + (long long)row * a.dv : nullptr;
  float* segst = segmented ? a.seg_state + (seg_at + head0 + mh) * hs + (long long)row * a.dv : nullptr;
  float S[32];
  {
    const float* init = nullptr;
    if (!STATE_ONLY) {
      if (segmented) init = segst;
      else if (a.starts[seq] != 0) init = cache;
    }
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
      const float4 v = init != nullptr && row < a.dk && mc + i < a.dv ? *reinterpret_cast<const float4*>(init + mc + i)
                                                                     : make_float4(0.f, 0.f, 0.f, 0.f);
      S[i] = v.x; S[i + 1] = v.y; S[i + 2] = v.z; S[i + 3] = v.w;
    }
  }

  // 16-byte unit n of mine where tiles are worked on row by row: row urow + 32 n, unit tid & 15
  const int cu8 = (tid & 15) * 8, urow = tid >> 4;
  const int uh = NH == 2 ? cu8 >> 6 : 0, uc = NH == 2 ? cu8 & 63 : c0 + cu8;     // as value columns: a head and its columns

  const float skip = a.skip != nullptr ? a.skip[head0 + mh] : 0.f;
  float log_sum = 0.f;                                        // (STATE_ONLY) log2 decay over the segment
  bool ok = true;
  uint32_t phase = 0;
  int chunk = 0;
  for (; chunk < n_chunk; ++chunk, phase ^= 1u) {
    const int buf = chunk & 1;
    const bool more = chunk + 1 < n_chunk;
    const uint32_t sK = sK0 + (uint32_t)buf * TILE;
    const uint32_t kphase = (uint32_t)(chunk >> 1) & 1u;
    auto k_full = [&] { return mbar_wait(full_k + (uint32_t)buf * 8u, kphase); };

    // v' = weight * v of the units of mine, high and low part, to the state's tiles
    auto put_weighted = [&]() {
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const uint32_t off = tile_off(urow + 32 * n, tid & 15);
        const float w1 = sm.wk[buf][uh][urow + 32 * n];
        const float2 w = make_float2(w1, w1);
        const uint4 v = ld_shared(sV + off);
        uint4 h, l;
        split2(fmul2(unpack2(v.x), w), h.x, l.x);
        split2(fmul2(unpack2(v.y), w), h.y, l.y);
        split2(fmul2(unpack2(v.z), w), h.z, l.z);
        split2(fmul2(unpack2(v.w), w), h.w, l.w);
        st_shared(sSh + off, h);
        st_shared(sSl + off, l);
      }
    };
    auto put_norm_sums = [&]() {                              // what the chunk adds to n, by warp
      float2 add[4] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const float w1 = sm.wk[buf][0][urow + 32 * n];
        const float2 w = make_float2(w1, w1);
        const uint4 k = ld_shared(sK + tile_off(urow + 32 * n, tid & 15));
        add[0] = ffma2(unpack2(k.x), w, add[0]);
        add[1] = ffma2(unpack2(k.y), w, add[1]);
        add[2] = ffma2(unpack2(k.z), w, add[2]);
        add[3] = ffma2(unpack2(k.w), w, add[3]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        add[i].x += __shfl_xor_sync(0xffffffffu, add[i].x, 16);
        add[i].y += __shfl_xor_sync(0xffffffffu, add[i].y, 16);
        if (lane < 16) *reinterpret_cast<float2*>(&sm.n_add[warp][cu8 + 2 * i]) = add[i];
      }
    };
    auto advance_norm = [&]() {
      if (tid < N) {
        float v = sm.n[tid] * fast_exp2(sm.dec[buf][0]);
#pragma unroll
        for (int w = 0; w < kThreads / 32; ++w) v += sm.n_add[w][tid];
        sm.n[tid] = v;
      }
    };
    const uint64_t khd = smem_desc(sK, SLAB, 1024), shd = smem_desc(sSh, SLAB, 1024), sld = smem_desc(sSl, SLAB, 1024);
    auto issue_state = [&]() {
#pragma unroll
      for (int ks = 0; ks < 8; ++ks) {
        tc_mma_ss(tmem + 384u, khd + (uint64_t)(ks * 128), shd + (uint64_t)(ks * 128), IDESC_AB, ks > 0 ? 1u : 0u);
        tc_mma_ss(tmem + 384u, khd + (uint64_t)(ks * 128), sld + (uint64_t)(ks * 128), IDESC_AB, 1u);
      }
      tc_commit(bar_s);
    };

    // ---- the state's tiles: S, or (STATE_ONLY) V' at once ------------------------------------------------
    if constexpr (STATE_ONLY) {
      ok = mbar_wait(full_v, phase) && ok;
      ok = k_full() && ok;
      put_weighted();
      if constexpr (NORM) put_norm_sums();
    } else {
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        uint4 h, l;
        split2(make_float2(S[8 * u], S[8 * u + 1]), h.x, l.x);
        split2(make_float2(S[8 * u + 2], S[8 * u + 3]), h.y, l.y);
        split2(make_float2(S[8 * u + 4], S[8 * u + 5]), h.z, l.z);
        split2(make_float2(S[8 * u + 6], S[8 * u + 7]), h.w, l.w);
        const uint32_t off = tile_off(row, cg * 4 + u);
        st_shared(sSh + off, h);
        st_shared(sSl + off, l);
      }
    }
    fence_proxy_async();
    tc_fence_before();                                        // the last chunk's tensor-memory reads are done
    __syncthreads();
    if (warp == 0) {
      if constexpr (!STATE_ONLY) ok = mbar_wait(full_q, phase) && ok;
      ok = k_full() && ok;
      tc_fence_after();
      __syncwarp();
      if constexpr (STATE_ONLY) {
        issue_state();
      } else {
        const uint64_t qd = smem_desc(sQ, 16, 1024), kd = smem_desc(sK, 16, 1024);
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {
          const uint32_t off = (uint32_t)(ks >> 2) * (SLAB >> 4) + (uint32_t)(ks & 3) * 2u;
          tc_mma_ss(tmem, qd + off, kd + off, IDESC_QK, ks > 0 ? 1u : 0u);
        }
        tc_commit(bar_a);
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {
          const uint32_t off = (uint32_t)(ks >> 2) * (SLAB >> 4) + (uint32_t)(ks & 3) * 2u;
          tc_mma_ss(tmem + 128u, qd + off, shd + (uint64_t)(ks * 128), IDESC_B, ks > 0 ? 1u : 0u);
          tc_mma_ss(tmem + 128u, qd + off, sld + (uint64_t)(ks * 128), IDESC_B, 1u);
        }
        tc_commit(bar_1);
      }
    }
    if (copier) {
      if (more) { load_k(chunk + 1); ++n_k; }                 // (its last readers were done before the last chunk's end)
      if (!STATE_ONLY && chunk > 0) {                         // the output has left V's place
        tma_store_wait_read();
        load_v(chunk);
        ++n_v;
      }
      if (STATE_ONLY && more) { load_v(chunk + 1); ++n_v; }   // V has become V'
    }
    __syncwarp();
    if (warp < NH && more) fetch_gates(chunk + 1);
    if constexpr (!STATE_ONLY) {
      float floor = 0.f, den = 0.f;
      if constexpr (NORM) {
        const long long t = t0 + (long long)chunk * C + row;
        if (t < t1) floor = a.floor[(long long)head0 * a.total + t];
        ok = mbar_wait(full_q, phase) && ok;
        ok = k_full() && ok;
        put_norm_sums();
        float2 d2 = make_float2(0.f, 0.f);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const uint4 q = ld_shared(sQ + tile_off(row, cg * 4 + u));
          const float4 n0 = *reinterpret_cast<const float4*>(sm.n + cg * 32 + u * 8), n1 = *reinterpret_cast<const float4*>(sm.n + cg * 32 + u * 8 + 4);
          d2 = ffma2(unpack2(q.x), make_float2(n0.x, n0.y), d2);
          d2 = ffma2(unpack2(q.y), make_float2(n0.z, n0.w), d2);
          d2 = ffma2(unpack2(q.z), make_float2(n1.x, n1.y), d2);
          d2 = ffma2(unpack2(q.w), make_float2(n1.z, n1.w), d2);
        }
        den = (d2.x + d2.y) * fast_exp2(sm.lb[buf][0][row].x);
      }
      // ---- A -> P ------------------------------------------------------------------------------------
      ok = mbar_wait(bar_a, phase) && ok;
      tc_fence_after();
      float s[32];
      tc_ld32(tA, s);
      tc_wait_ld();
      tc_fence_before();
      __syncthreads();                                        // P is written over other warps' part of A; n has been read
      tc_fence_after();
      if constexpr (NORM) advance_norm();
      const int over = row - cg * 32;                         // my columns up to this one are at or before my row
      const bool below = __any_sync(0xffffffffu, over >= 0);
#pragma unroll
      for (int hh = 0; hh < NH; ++hh) {
        const float2* lb = sm.lb[buf][hh] + cg * 32;
        const float li = sm.lb[buf][hh][row].x;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          uint32_t ph[8], pl[8];
          if (below) {
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              const int j = h * 16 + 2 * i;
              const float4 w = *reinterpret_cast<const float4*>(lb + j);
              const float2 e = make_float2(fast_exp2(li - w.x), fast_exp2(li - w.z));
              float2 p = fmul2(make_float2(s[j], s[j + 1]), fmul2(e, make_float2(w.y, w.w)));
              p.x = j <= over ? p.x : 0.f;                    // (a selection: what is dropped may have overflowed)
              p.y = j + 1 <= over ? p.y : 0.f;
              if constexpr (NORM) den += p.x + p.y;
              split2(p, ph[i], pl[i]);
            }
          } else {
#pragma unroll
            for (int i = 0; i < 8; ++i) ph[i] = pl[i] = 0u;
          }
          tc_st8(tP + hh * 384u + h * 8u, ph);
          tc_st8(tP + hh * 384u + 64u + h * 8u, pl);
        }
      }
      if constexpr (NORM) sm.den[cg][row] = den;
      tc_wait_st();
      tc_fence_before();
      __syncthreads();
      if (warp == 0) {
        ok = mbar_wait(full_v, phase) && ok;
        tc_fence_after();
        __syncwarp();
        const uint64_t vd = smem_desc(sV, SLAB, 1024);
#pragma unroll
        for (int hh = 0; hh < NH; ++hh) {
          const uint64_t vh = vd + (uint64_t)(hh * (SLAB >> 4));
          const uint32_t d = tmem + 256u + (uint32_t)hh * 64u, p = tmem + (uint32_t)hh * 384u;
#pragma unroll
          for (int ks = 0; ks < 8; ++ks) {
            tc_mma_ts(d, p + (uint32_t)ks * 8u, vh + (uint64_t)(ks * 128), IDESC_PV, ks > 0 ? 1u : 0u);
            tc_mma_ts(d, p + 64u + (uint32_t)ks * 8u, vh + (uint64_t)(ks * 128), IDESC_PV, 1u);
          }
        }
        tc_commit(bar_o);
      }
      // ---- V' over the state's tiles ----------------------------------------------------------------
      ok = mbar_wait(bar_1, phase) && ok;
      ok = mbar_wait(full_v, phase) && ok;
      if (copier && more) { load_q(chunk + 1); ++n_q; }
      __syncwarp();
      put_weighted();
      fence_proxy_async();
      __syncthreads();
      if (warp == 0) {                                        // (in order behind the products that read the second head's P there)
        tc_fence_after();
        __syncwarp();
        issue_state();
      }
      // ---- output, over V --------------------------------------------------------------------------------
      const float e = fast_exp2(sm.lb[buf][mh][row].x) * a.q_scale;
      float f2 = a.q_scale, f1 = e;
      if constexpr (NORM) {
        const float dn = a.q_scale * (sm.den[0][row] + sm.den[1][row] + sm.den[2][row] + sm.den[3][row]);
        const float inv = 1.f / (fmaxf(fabsf(dn), floor) + a.norm_eps);
        f1 *= inv;
        f2 *= inv;
      }
      ok = mbar_wait(bar_o, phase) && ok;
      tc_fence_after();
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        float x[16], y[16];
        tc_ld16(tO1 + h * 16u, x);
        tc_ld16(tO2 + h * 16u, y);
        tc_wait_ld();
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const uint32_t off = tile_off(row, cg * 4 + h * 2 + u);
          uint32_t p[4];
          uint4 vu = make_uint4(0, 0, 0, 0);
          if (!NORM) vu = ld_shared(sV + off);
          const uint32_t vv[4] = {vu.x, vu.y, vu.z, vu.w};
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int j = u * 8 + 2 * i;
            float2 r = ffma2(make_float2(x[j], x[j + 1]), make_float2(f1, f1), fmul2(make_float2(y[j], y[j + 1]), make_float2(f2, f2)));
            if (!NORM) r = ffma2(unpack2(vv[i]), make_float2(skip, skip), r);
            p[i] = pack_bf162(r.x, r.y);
          }
          st_shared(sV + off, make_uint4(p[0], p[1], p[2], p[3]));
        }
      }
      fence_proxy_async();
    } else {
      if constexpr (NORM) advance_norm();
    }
    // ---- state ---------------------------------------------------------------------------------------
    ok = mbar_wait(bar_s, phase) && ok;
    tc_fence_after();
    {
      const float ld = sm.dec[buf][mh], dc = fast_exp2(ld);
      if (STATE_ONLY) log_sum += ld;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        float t[16];
        tc_ld16(tS + h * 16u, t);
        tc_wait_ld();
#pragma unroll
        for (int i = 0; i < 16; i += 2) {
          const float2 r = ffma2(make_float2(S[h * 16 + i], S[h * 16 + i + 1]), make_float2(dc, dc), make_float2(t[i], t[i + 1]));
          S[h * 16 + i] = r.x;
          S[h * 16 + i + 1] = r.y;
        }
      }
    }
    if (warp < NH && more) put_gates(buf ^ 1);
    if (__syncthreads_or(ok ? 0 : 1)) break;                  // a wait ran out somewhere in the CTA
    if constexpr (!STATE_ONLY) {
      const int rows = n_tok - chunk * C;
      const long long tb = t0 + (long long)chunk * C;
      if (rows >= C) {
        if (copier) {
          if (NH == 2) {
            tma_store_3d(&omap, 0, head0, (int)tb, sV);
            tma_store_3d(&omap, 0, head0 + 1, (int)tb, sV + SLAB);
          } else {
            tma_store_3d(&omap, c0, head0, (int)tb, sV);
            if (wide_v) tma_store_3d(&omap, c0 + 64, head0, (int)tb, sV + SLAB);
          }
          tma_store_commit();
        }
        __syncwarp();
      } else {                                                // the last chunk of a sequence: its rows only
        bf16* p = static_cast<bf16*>(a.out) + (tb + urow) * ((long long)a.heads * a.dv) + (long long)(head0 + uh) * a.dv + uc;
#pragma unroll
        for (int n = 0; n < 4; ++n)
          if (uc < a.dv && urow + 32 * n < rows)
            *reinterpret_cast<uint4*>(p + (long long)(32 * n) * a.heads * a.dv) = ld_shared(sV + tile_off(urow + 32 * n, tid & 15));
      }
    }
  }
  if (chunk < n_chunk) {                                      // left early: wait (bounded) for what is still in flight
    if (tid == 0) atomicOr(a.status, kStatusWaitTimeout);
    if (!STATE_ONLY) {
      mbar_wait(bar_a, phase);
      mbar_wait(bar_1, phase);
      mbar_wait(bar_o, phase);
    }
    mbar_wait(bar_s, phase);
  }
  if (copier) {                                               // copies into and out of this CTA's shared memory
    if (n_q > 0) mbar_wait(full_q, (uint32_t)(n_q - 1) & 1u);
    if (n_k > 0) mbar_wait(full_k + (uint32_t)((n_k - 1) & 1) * 8u, (uint32_t)((n_k - 1) >> 1) & 1u);
    if (n_v > 0) mbar_wait(full_v, (uint32_t)(n_v - 1) & 1u);
    tma_store_wait_read();
  }
  __syncwarp();
  float* dst = STATE_ONLY ? segst : (last_seg ? cache : nullptr);
  if (dst != nullptr && row < a.dk) {
#pragma unroll
    for (int i = 0; i < 32; i += 4)
      if (mc + i < a.dv) *reinterpret_cast<float4*>(dst + mc + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
  }
  if (STATE_ONLY && blockIdx.z == 0 && row == 0 && (NH == 2 ? (cg & 1) == 0 : cg == 0)) a.seg_log[seg_at + head0 + mh] = log_sum;
  if (NORM && blockIdx.z == 0 && tid < a.dk) {
    if (STATE_ONLY) a.seg_norm[(seg_at + head0) * a.dk + tid] = sm.n[tid];
    else if (last_seg && slot_ok)
      a.norm[(((long long)slot * 2 + ((a.starts[seq] + seq_len - 1) & 1)) * a.heads + head0) * a.dk + tid] = sm.n[tid];
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    __syncwarp();
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
  }
}

// seg_state[seq, s] (and seg_norm) holds what segment s adds; turned in place into the state at the start of segment s.
__global__ void __launch_bounds__(256) recurrence_segment_scan_kernel(const RecurrenceArgs a) {
  const long long hs = (long long)a.dk * a.dv;
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  const int head = blockIdx.y, seq = blockIdx.z;
  const bool norm = i >= hs;
  if (i >= hs + (a.floor != nullptr ? a.dk : 0)) return;
  const long long n = a.cu[seq + 1] - (long long)a.cu[seq];
  const int n_seg = (int)((n + a.seg_len - 1) / a.seg_len);
  const int slot = a.slots[seq];
  float s = 0.f;
  if (norm) s = a.n0[((long long)seq * a.heads + head) * a.dk + i - hs];
  else if (a.starts[seq] != 0 && slot >= 0 && slot < a.n_slots) s = a.state[((long long)slot * a.heads + head) * hs + i];
  const long long at = (long long)seq * a.max_segs * a.heads + head;
  float* p = norm ? a.seg_norm + at * a.dk + i - hs : a.seg_state + at * hs + i;
  const long long step = (long long)a.heads * (norm ? a.dk : hs);
  const float* lg = a.seg_log + at;
  for (int k = 0; k < n_seg && k < a.max_segs; ++k, p += step, lg += a.heads) {
    const bool more = k + 1 < n_seg;                // the last segment's slot was not written
    const float add = more ? *p : 0.f;
    *p = s;
    s = more ? fast_exp2(*lg) * s + add : s;
  }
}

// Heads per CTA.
int tile_heads(int heads, int kv_rep, int dv, bool norm) { return !norm && dv <= 64 && kv_rep % 2 == 0 && heads % 2 == 0 ? 2 : 1; }

template <int NH, bool NORM>
cudaError_t launch_t(const RecurrenceArgs& a, EncodeTiledFn enc, cudaStream_t stream) {
  const dim3 grid((unsigned)(a.n_seq * a.max_segs), (unsigned)(a.heads / NH), (unsigned)((a.dv + N - 1) / N));
  const auto* x = static_cast<const bf16*>(a.qkv);
  const int groups = a.heads / a.kv_rep;
  CUtensorMap qmap, kmap, vmap, omap;
  if (!make_map3(enc, &qmap, x + a.off_q, a.dk, groups, a.total, a.dk, a.stride) ||
      !make_map3(enc, &kmap, x + a.off_k, a.dk, groups, a.total, a.dk, a.stride) ||
      !make_map3(enc, &vmap, x + a.off_v, a.dv, a.heads, a.total, a.dv, a.stride) ||
      !make_map3(enc, &omap, a.out, a.dv, a.heads, a.total, a.dv, (long long)a.heads * a.dv))
    return cudaErrorInvalidValue;
  cudaError_t e;
  if (a.max_segs > 1) {
    e = cudaFuncSetAttribute(recurrence_tc5_kernel<true, NH, NORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (e != cudaSuccess) return e;
    recurrence_tc5_kernel<true, NH, NORM><<<grid, kThreads, kSmem, stream>>>(qmap, kmap, vmap, omap, a);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    const long long n = (long long)a.dk * a.dv + (NORM ? a.dk : 0);
    recurrence_segment_scan_kernel<<<dim3((unsigned)((n + 255) / 256), (unsigned)a.heads, (unsigned)a.n_seq), 256, 0, stream>>>(a);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
  }
  e = cudaFuncSetAttribute(recurrence_tc5_kernel<false, NH, NORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
  if (e != cudaSuccess) return e;
  recurrence_tc5_kernel<false, NH, NORM><<<grid, kThreads, kSmem, stream>>>(qmap, kmap, vmap, omap, a);
  return cudaGetLastError();
}

}  // namespace

int recurrence_segments(int n_seq, int heads, int kv_rep, int dk, int dv, int max_len, int sm_count, int* seg_len) {
  // one CTA per SM, in segments of at least 512 tokens: a segment's keys and values are read twice, which only pays while SMs
  // would stay empty.  (Heads with a normaliser never share a CTA; counting them as if they did only makes more segments.)
  (void)dk;
  const int nh = tile_heads(heads, kv_rep, dv, false);
  const long long tasks = (long long)n_seq * (heads / nh) * ((dv + N - 1) / N);
  const long long segs = tasks * 2 > sm_count ? 1 : sm_count / tasks;
  long long len = (max_len + segs - 1) / segs;
  if (len < 512) len = 512;
  len = (len + C - 1) / C * C;
  *seg_len = (int)len;
  return (int)((max_len + len - 1) / len);
}

bool recurrence_tc5_supported(const RecurrenceArgs& a) {
  return a.cu != nullptr && a.dk <= N && a.dk % 8 == 0 && a.dv % 8 == 0 && a.stride % 8 == 0 && a.off_q % 8 == 0 && a.off_k % 8 == 0 &&
         a.off_v % 8 == 0 && (reinterpret_cast<uintptr_t>(a.qkv) & 15) == 0 && (reinterpret_cast<uintptr_t>(a.out) & 15) == 0 &&
         (reinterpret_cast<uintptr_t>(a.state) & 15) == 0 && (a.floor == nullptr || a.skip == nullptr);
}

cudaError_t launch_recurrence_tc5(const RecurrenceArgs& a, void* encode_fn, cudaStream_t stream) {
  if (a.n_seq == 0) return cudaSuccess;
  EncodeTiledFn enc = reinterpret_cast<EncodeTiledFn>(encode_fn);
  if (a.floor != nullptr) return launch_t<1, true>(a, enc, stream);
  return tile_heads(a.heads, a.kv_rep, a.dv, false) == 2 ? launch_t<2, false>(a, enc, stream) : launch_t<1, false>(a, enc, stream);
}

}  // namespace mixers
}  // namespace fa
