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
// Shared memory: five tiles of 128 x 128 bfloat16 (Q, K, V, and S high and low, whose place V' takes once O1 is done), each two
// 128-byte-swizzled slabs of 64 columns.  Waits are bounded: one that runs out sets the status word and the CTA leaves after another
// bounded wait for its MMAs.
#include "../hybrid/hybrid_common.cuh"
#include "../tc5.cuh"
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
  uint64_t bars[4];
  uint32_t tmem_slot;
};
constexpr int kSmem = 1024 + 5 * TILE + (int)sizeof(Small);
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
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf162(x, y);
  const float2 r = unpack2(hi);
  lo = pack_bf162(x - r.x, y - r.y);
}

template <bool STATE_ONLY, int NH, bool NORM>
__global__ void __launch_bounds__(kThreads, 1) recurrence_tc5_kernel(const RecurrenceArgs a) {
  static_assert(NH == 1 || !NORM, "a pair of heads has no normaliser");
  // instruction descriptors: fp32 accumulators, bfloat16 operands, M = 128, N at bit 17; bit 15: A MN-major, bit 16: B MN-major
  constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(128 >> 4) << 24);
  constexpr uint32_t N128 = (uint32_t)(N >> 3) << 17, NPV = (uint32_t)((N / NH) >> 3) << 17;
  constexpr uint32_t IDESC_QK = IDESC | N128, IDESC_B = IDESC | N128 | (1u << 16), IDESC_PV = IDESC | NPV | (1u << 16),
                     IDESC_AB = IDESC | N128 | (1u << 15) | (1u << 16);
  extern __shared__ uint8_t smem_dyn[];
  const uint32_t raw_base = smem_u32(smem_dyn);
  uint8_t* smem = smem_dyn + ((1024u - (raw_base & 1023u)) & 1023u);
  const uint32_t sQ = smem_u32(smem), sK = sQ + TILE, sV = sK + TILE, sSh = sV + TILE, sSl = sSh + TILE;
  Small& sm = *reinterpret_cast<Small*>(smem + 5 * TILE);
  const uint32_t bar_a = smem_u32(&sm.bars[0]), bar_1 = smem_u32(&sm.bars[1]), bar_o = smem_u32(&sm.bars[2]), bar_s = smem_u32(&sm.bars[3]);

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

  if (tid == 0) {
    for (int i = 0; i < 4; ++i) mbar_init(smem_u32(&sm.bars[i]), 1);
    mbar_fence_init();
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
      gl[i] = in ? a.la[at + i] * kLog2e : 0.f;
      gb[i] = in ? a.b[at + i] : 0.f;
    }
  };
  auto put_gates = [&](int buf) {
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

  // ---- fetching: four 16-byte units of each of q, k and v per thread --------------------------------
  const bf16* base = static_cast<const bf16*>(a.qkv);
  const int cu8 = (tid & 15) * 8, urow = tid >> 4;           // unit n of mine: row urow + 32 n, columns cu8 .. + 7
  const int uh = NH == 2 ? cu8 >> 6 : 0, uc = NH == 2 ? cu8 & 63 : c0 + cu8;     // as value columns: a head and its columns
  const bool k_ok = cu8 < a.dk, v_ok = uc < a.dv;
  const int v_col = (head0 + uh) * a.dv + uc;
  uint4 rq[STATE_ONLY ? 1 : 4], rk[4], rv[4];
  auto fetch = [&](int chunk) {
    const long long tb = t0 + (long long)chunk * C + urow;
    const bf16* p = base + tb * a.stride;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const bool in = tb + 32 * n < t1;
      const bf16* pr = p + (long long)(32 * n) * a.stride;
      const uint4 z = make_uint4(0, 0, 0, 0);
      if (!STATE_ONLY) rq[n] = in && k_ok ? *reinterpret_cast<const uint4*>(pr + a.off_q + grp * a.dk + cu8) : z;
      rk[n] = in && k_ok ? *reinterpret_cast<const uint4*>(pr + a.off_k + grp * a.dk + cu8) : z;
      rv[n] = in && v_ok ? *reinterpret_cast<const uint4*>(pr + a.off_v + v_col) : z;
    }
  };
  // the rows that fetch() will read, on their way to the L2 while the current chunk is computed
  auto prefetch = [&](int chunk) {
    const long long tb = t0 + (long long)chunk * C + urow;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      if (tb + 32 * n < t1 && (tid & 7) == 0) {
        const bf16* pr = base + (tb + 32 * n) * a.stride;
        if (!STATE_ONLY && k_ok) asm volatile("prefetch.global.L2 [%0];" ::"l"(pr + a.off_q + grp * a.dk + cu8));
        if (k_ok) asm volatile("prefetch.global.L2 [%0];" ::"l"(pr + a.off_k + grp * a.dk + cu8));
        if (v_ok) asm volatile("prefetch.global.L2 [%0];" ::"l"(pr + a.off_v + v_col));
      }
    }
  };
  // The finished chunk's output lies in the Q tile; every thread stores the units it will overwrite with the next queries.
  auto store_out = [&](int done) {
    const long long tb = t0 + (long long)done * C + urow;
    bf16* p = static_cast<bf16*>(a.out) + tb * ((long long)a.heads * a.dv) + v_col;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const uint4 v = ld_shared(sQ + tile_off(urow + 32 * n, tid & 15));
      if (v_ok && tb + 32 * n < t1) *reinterpret_cast<uint4*>(p + (long long)(32 * n) * a.heads * a.dv) = v;
    }
  };

  const float skip = a.skip != nullptr ? a.skip[head0 + mh] : 0.f;
  float log_sum = 0.f;                                        // (STATE_ONLY) log2 decay over the segment
  bool ok = true;
  uint32_t phase = 0;
  fetch(0);
  int chunk = 0;
  for (; chunk < n_chunk; ++chunk, phase ^= 1u) {
    const int buf = chunk & 1;
    if (chunk + 1 < n_chunk) prefetch(chunk + 1);
    if (!STATE_ONLY && chunk > 0) store_out(chunk - 1);
    // ---- tiles ----------------------------------------------------------------------------------------
    if constexpr (NORM) {                                     // what the chunk adds to n
      float add[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const float w = sm.wk[buf][0][urow + 32 * n];
        const uint32_t k[4] = {rk[n].x, rk[n].y, rk[n].z, rk[n].w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 f = unpack2(k[i]);
          add[2 * i] += w * f.x;
          add[2 * i + 1] += w * f.y;
        }
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) add[i] += __shfl_xor_sync(0xffffffffu, add[i], 16);
      if (lane < 16) {
#pragma unroll
        for (int i = 0; i < 8; ++i) sm.n_add[warp][cu8 + i] = add[i];
      }
    }
    // v' of a unit, high and low part
    auto weighted = [&](const uint4& v, int r, uint4& h, uint4& l) {
      const float w = sm.wk[buf][uh][r];
      float2 f;
      f = unpack2(v.x); split2(f.x * w, f.y * w, h.x, l.x);
      f = unpack2(v.y); split2(f.x * w, f.y * w, h.y, l.y);
      f = unpack2(v.z); split2(f.x * w, f.y * w, h.z, l.z);
      f = unpack2(v.w); split2(f.x * w, f.y * w, h.w, l.w);
    };
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const uint32_t off = tile_off(urow + 32 * n, tid & 15);
      st_shared(sK + off, rk[n]);
      if constexpr (!STATE_ONLY) {
        st_shared(sQ + off, rq[n]);
        st_shared(sV + off, rv[n]);
      } else {
        uint4 h, l;
        weighted(rv[n], urow + 32 * n, h, l);
        st_shared(sSh + off, h);
        st_shared(sSl + off, l);
      }
    }
    if constexpr (!STATE_ONLY) {
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        uint4 h, l;
        split2(S[8 * u], S[8 * u + 1], h.x, l.x);
        split2(S[8 * u + 2], S[8 * u + 3], h.y, l.y);
        split2(S[8 * u + 4], S[8 * u + 5], h.z, l.z);
        split2(S[8 * u + 6], S[8 * u + 7], h.w, l.w);
        const uint32_t off = tile_off(row, cg * 4 + u);
        st_shared(sSh + off, h);
        st_shared(sSl + off, l);
      }
    }
    fence_proxy_async();
    tc_fence_before();                                        // the last chunk's tensor-memory reads are done
    __syncthreads();
    const uint64_t khd = smem_desc(sK, SLAB, 1024), shd = smem_desc(sSh, SLAB, 1024), sld = smem_desc(sSl, SLAB, 1024);
    auto issue_state = [&]() {
#pragma unroll
      for (int ks = 0; ks < 8; ++ks) {
        tc_mma_ss(tmem + 384u, khd + (uint64_t)(ks * 128), shd + (uint64_t)(ks * 128), IDESC_AB, ks > 0 ? 1u : 0u);
        tc_mma_ss(tmem + 384u, khd + (uint64_t)(ks * 128), sld + (uint64_t)(ks * 128), IDESC_AB, 1u);
      }
      tc_commit(bar_s);
    };
    if (warp == 0) {
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
    if (warp < NH && chunk + 1 < n_chunk) fetch_gates(chunk + 1);
    if constexpr (!STATE_ONLY) {
      float floor = 0.f, den = 0.f;
      if constexpr (NORM) {
        const long long t = t0 + (long long)chunk * C + row;
        if (t < t1) floor = a.floor[(long long)head0 * a.total + t];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const uint4 q = ld_shared(sQ + tile_off(row, cg * 4 + u));
          const float* n = sm.n + cg * 32 + u * 8;
          float2 f;
          f = unpack2(q.x); den += f.x * n[0] + f.y * n[1];
          f = unpack2(q.y); den += f.x * n[2] + f.y * n[3];
          f = unpack2(q.z); den += f.x * n[4] + f.y * n[5];
          f = unpack2(q.w); den += f.x * n[6] + f.y * n[7];
        }
        den *= fast_exp2(sm.lb[buf][0][row].x);
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
      if constexpr (NORM) {
        if (tid < N) {
          float v = sm.n[tid] * fast_exp2(sm.dec[buf][0]);
#pragma unroll
          for (int w = 0; w < kThreads / 32; ++w) v += sm.n_add[w][tid];
          sm.n[tid] = v;
        }
      }
      const bool below = cg * 32 <= (warp & 3) * 32 + 31;     // some of my columns are at or before some of my rows
#pragma unroll
      for (int hh = 0; hh < NH; ++hh) {
        const float2* lb = sm.lb[buf][hh] + cg * 32;
        const float li = sm.lb[buf][hh][row].x;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          uint32_t ph[8], pl[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const int j = h * 16 + 2 * i;
            float x = 0.f, y = 0.f;
            if (below) {
              const float4 w = *reinterpret_cast<const float4*>(lb + j);
              if (cg * 32 + j <= row) x = s[j] * (w.y * fast_exp2(li - w.x));
              if (cg * 32 + j + 1 <= row) y = s[j + 1] * (w.w * fast_exp2(li - w.z));
            }
            if constexpr (NORM) den += x + y;
            split2(x, y, ph[i], pl[i]);
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
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const uint32_t off = tile_off(urow + 32 * n, tid & 15);
        uint4 h, l;
        weighted(ld_shared(sV + off), urow + 32 * n, h, l);          // (a unit that this thread has written)
        st_shared(sSh + off, h);
        st_shared(sSl + off, l);
      }
      fence_proxy_async();
      if constexpr (NH == 2) ok = mbar_wait(bar_o, phase) && ok;     // dS takes the place of the second head's P
      __syncthreads();
      if (warp == 0) {
        tc_fence_after();
        __syncwarp();
        issue_state();
      }
      if (chunk + 1 < n_chunk) fetch(chunk + 1);
      // ---- output ------------------------------------------------------------------------------------
      ok = mbar_wait(bar_o, phase) && ok;
      tc_fence_after();
      const float e = fast_exp2(sm.lb[buf][mh][row].x) * a.q_scale;
      float f2 = a.q_scale, f1 = e;
      if constexpr (NORM) {
        const float dn = a.q_scale * (sm.den[0][row] + sm.den[1][row] + sm.den[2][row] + sm.den[3][row]);
        const float inv = 1.f / (fmaxf(fabsf(dn), floor) + a.norm_eps);
        f1 *= inv;
        f2 *= inv;
      }
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
          if (!NORM) {
            const uint4 vu = ld_shared(sV + off);
            const uint32_t vv[4] = {vu.x, vu.y, vu.z, vu.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const float2 v = unpack2(vv[i]);
              const int j = u * 8 + 2 * i;
              p[i] = pack_bf162(f1 * x[j] + f2 * y[j] + skip * v.x, f1 * x[j + 1] + f2 * y[j + 1] + skip * v.y);
            }
          } else {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const int j = u * 8 + 2 * i;
              p[i] = pack_bf162(f1 * x[j] + f2 * y[j], f1 * x[j + 1] + f2 * y[j + 1]);
            }
          }
          st_shared(sQ + off, make_uint4(p[0], p[1], p[2], p[3]));   // Q is no longer read
        }
      }
    } else {
      if (chunk + 1 < n_chunk) fetch(chunk + 1);
      if constexpr (NORM) {
        if (tid < N) {
          float v = sm.n[tid] * fast_exp2(sm.dec[buf][0]);
#pragma unroll
          for (int w = 0; w < kThreads / 32; ++w) v += sm.n_add[w][tid];
          sm.n[tid] = v;
        }
      }
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
        for (int i = 0; i < 16; ++i) S[h * 16 + i] = dc * S[h * 16 + i] + t[i];
      }
    }
    if (warp < NH && chunk + 1 < n_chunk) put_gates(buf ^ 1);
    if (__syncthreads_or(ok ? 0 : 1)) break;                  // a wait ran out somewhere in the CTA
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
  if (!STATE_ONLY && chunk == n_chunk) store_out(n_chunk - 1);
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
cudaError_t launch_t(const RecurrenceArgs& a, cudaStream_t stream) {
  const dim3 grid((unsigned)(a.n_seq * a.max_segs), (unsigned)(a.heads / NH), (unsigned)((a.dv + N - 1) / N));
  cudaError_t e;
  if (a.max_segs > 1) {
    e = cudaFuncSetAttribute(recurrence_tc5_kernel<true, NH, NORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (e != cudaSuccess) return e;
    recurrence_tc5_kernel<true, NH, NORM><<<grid, kThreads, kSmem, stream>>>(a);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
    const long long n = (long long)a.dk * a.dv + (NORM ? a.dk : 0);
    recurrence_segment_scan_kernel<<<dim3((unsigned)((n + 255) / 256), (unsigned)a.heads, (unsigned)a.n_seq), 256, 0, stream>>>(a);
    e = cudaGetLastError();
    if (e != cudaSuccess) return e;
  }
  e = cudaFuncSetAttribute(recurrence_tc5_kernel<false, NH, NORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
  if (e != cudaSuccess) return e;
  recurrence_tc5_kernel<false, NH, NORM><<<grid, kThreads, kSmem, stream>>>(a);
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

cudaError_t launch_recurrence_tc5(const RecurrenceArgs& a, cudaStream_t stream) {
  if (a.n_seq == 0) return cudaSuccess;
  if (a.floor != nullptr) return launch_t<1, true>(a, stream);
  return tile_heads(a.heads, a.kv_rep, a.dv, false) == 2 ? launch_t<2, false>(a, stream) : launch_t<1, false>(a, stream);
}

}  // namespace mixers
}  // namespace fa
