// Decayed linear attention over prompts on the 5th-generation tensor cores (tcgen05 + TMEM), sm_100a: heads of up to 128
// key columns and any number of value columns.
//
// The arithmetic is that of lightning_chunk.cu (see there) with chunks of C = 128 tokens, the 128 lanes of tensor memory:
//     A  = Q K^T                      (128 x 128)            O1 = Q S          S enters as two bfloat16 parts
//     P  = A, decayed and masked, as two bfloat16 parts      O2 = P V          P is read from tensor memory, over A
//     o_i = d^(i+1) O1_i + O2_i                              dS = K'^T V       k'_j = d^(C-1-j) k_j, two bfloat16 parts
//     S  <- d^C S + dS                                       S stays in the threads' registers, fp32
// CTA = (segment of a sequence, head, 128 value columns), sixteen warps, all of them with the same role: a warp owns 32 lanes
// (rows) x 32 columns of whatever is in tensor memory; warp 0 issues the MMAs.
//
// Tensor memory, 512 columns: A / P [0, 128)  O1 [128, 256)  O2 [256, 384)  dS [384, 512).  Shared memory: seven tiles of
// 128 x 128 bfloat16 (Q, K, V, K' high, K' low, S high, S low), each two 128-byte-swizzled slabs of 64 columns.
// Waits are bounded: one that runs out sets the status word and the CTA leaves after another bounded wait for its MMAs.
#include "../tc5.cuh"
#include "hybrid_common.cuh"
#include "lightning.cuh"

namespace fa {
namespace hybrid {
namespace {

constexpr int C = 128;         // tokens per chunk
constexpr int N = 128;         // key and value columns per CTA (padded with zeros)
constexpr int kThreads = 512;
constexpr int SLAB = 128 * 128;
constexpr int TILE = 2 * SLAB;
constexpr int kSmem = 1024 + 7 * TILE + (2 * C + 4) * 4 + 4 * 8 + 16;
static_assert(kSmem <= 227 * 1024, "shared memory plan exceeds the SM");

// Byte offset of 16-byte unit `u` (0..15) of row `row` in a tile.
__device__ __forceinline__ uint32_t tile_off(int row, int u) {
  return (uint32_t)((u >> 3) * SLAB + row * 128 + ((u ^ row) & 7) * 16);
}
__device__ __forceinline__ void st_shared(uint32_t addr, const uint4& v) {
  asm volatile("st.shared.v4.b32 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(v.x), "r"(v.y), "r"(v.z), "r"(v.w) : "memory");
}
__device__ __forceinline__ float2 unpack2(uint32_t v) {
  return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u));
}
// SiLU of a pair with the hardware's exponential and ONE reciprocal, 1 / (ab) (the special function unit is what the activation
// waits for); all errors are far below the bfloat16 rounding that follows.  Below -40 the sigmoid stays at its value there,
// 4e-18, which keeps the product finite.
__device__ __forceinline__ uint32_t silu2(uint32_t raw) {
  const float2 z = unpack2(raw);
  const float a = 1.f + fast_exp2(-1.4426950408889634f * fmaxf(z.x, -40.f)), b = 1.f + fast_exp2(-1.4426950408889634f * fmaxf(z.y, -40.f));
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(a * b));
  return pack_bf162(z.x * (r * b), z.y * (r * a));
}
__device__ __forceinline__ uint4 silu8(const uint4& raw) {
  return make_uint4(silu2(raw.x), silu2(raw.y), silu2(raw.z), silu2(raw.w));
}
// Two fp32 numbers as packed (high, low) bfloat16 parts.
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf162(x, y);
  const float2 r = unpack2(hi);
  lo = pack_bf162(x - r.x, y - r.y);
}

template <bool STATE_ONLY>
__global__ void __launch_bounds__(kThreads, 1) lightning_tc5_kernel(const LightningArgs a) {
  // instruction descriptors: fp32 accumulators, bfloat16 operands, N = M = 128; bit 15: A MN-major, bit 16: B MN-major
  constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
  constexpr uint32_t IDESC_QK = IDESC, IDESC_B = IDESC | (1u << 16), IDESC_AB = IDESC | (1u << 15) | (1u << 16);
  extern __shared__ uint8_t smem_dyn[];
  const uint32_t raw_base = smem_u32(smem_dyn);
  uint8_t* smem = smem_dyn + ((1024u - (raw_base & 1023u)) & 1023u);
  const uint32_t sQ = smem_u32(smem), sK = sQ + TILE, sV = sK + TILE, sKh = sV + TILE, sKl = sKh + TILE, sSh = sKl + TILE, sSl = sSh + TILE;
  float* pz = reinterpret_cast<float*>(smem + 7 * TILE);               // [C] zeros, the weights of later tokens, then
  float* pw = pz + C;                                                  // decay^0 .. decay^C
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + 7 * TILE + (2 * C + 4) * 4);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 4);
  const uint32_t bar_a = smem_u32(bars), bar_s = smem_u32(bars + 1), bar_o = smem_u32(bars + 2);

  const int seq = blockIdx.x / a.max_segs, seg = blockIdx.x - seq * a.max_segs;
  const int head = blockIdx.y, c0 = blockIdx.z * N;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  long long t0 = a.cu[seq], t1 = a.cu[seq + 1];
  if (t0 < 0) t0 = 0;
  if (t1 > a.total) t1 = a.total;
  const long long seq_end = t1;
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
  float* cache = slot_ok ? a.state + ((long long)slot * a.heads + head) * hs : nullptr;
  float* segst = a.max_segs > 1 ? a.seg_state + (((long long)seq * a.max_segs + seg) * a.heads + head) * hs : nullptr;

  if (tid == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(smem_u32(bars + i), 1);
    mbar_fence_init();
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  {
    const float d = a.decay[head];
    for (int i = tid; i <= C; i += kThreads) {
      pw[i] = i == 0 ? 1.f : powf(d, (float)i);
      if (i < C) pz[i] = 0.f;
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  // my place in tensor memory: lane (row) and 32 columns
  const int row = (warp & 3) * 32 + lane, cg = warp >> 2;
  const uint32_t tl = tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)cg * 32u;
  const uint32_t tA = tl, tO1 = tl + 128u, tO2 = tl + 256u, tS = tl + 384u;
  const uint32_t tP = tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)cg * 16u;     // high part; low part 64 columns on

  // ---- state: row `row`, columns c0 + cg * 32 .. + 31 ---------------------------------------------
  float S[32];
  {
    const float* init = nullptr;
    if (!STATE_ONLY) {
      if (a.max_segs > 1) init = segst;
      else if (a.starts[seq] != 0) init = cache;
    }
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
      const int c = c0 + cg * 32 + i;
      const float4 v = init != nullptr && row < a.dk && c < a.dv ? *reinterpret_cast<const float4*>(init + (long long)row * a.dv + c)
                                                                : make_float4(0.f, 0.f, 0.f, 0.f);
      S[i] = v.x; S[i + 1] = v.y; S[i + 2] = v.z; S[i + 3] = v.w;
    }
  }

  // ---- fetching: four 16-byte units of each of q, k and v per thread --------------------------------
  const bf16* base = static_cast<const bf16*>(a.qkv);
  const int cu8 = (tid & 15) * 8, urow = tid >> 4;           // unit n of mine: row urow + 32 n, columns cu8 .. + 7
  const bool k_ok = cu8 < a.dk, v_ok = c0 + cu8 < a.dv;
  uint4 rq[STATE_ONLY ? 1 : 4], rk[4], rv[4];
  auto fetch = [&](int chunk) {
    const long long tb = t0 + (long long)chunk * C + urow;
    const bf16* p = base + tb * a.stride;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const bool in = tb + 32 * n < t1;
      const bf16* pr = p + (long long)(32 * n) * a.stride;
      const uint4 z = make_uint4(0, 0, 0, 0);
      if (!STATE_ONLY) rq[n] = in && k_ok ? *reinterpret_cast<const uint4*>(pr + a.off_q + head * a.dk + cu8) : z;
      rk[n] = in && k_ok ? *reinterpret_cast<const uint4*>(pr + a.off_k + head * a.dk + cu8) : z;
      rv[n] = in && v_ok ? *reinterpret_cast<const uint4*>(pr + a.off_v + head * a.dv + c0 + cu8) : z;
    }
  };

  // The finished chunk's output lies in the Q tile; every thread stores the units it will overwrite with the next queries.
  auto store_out = [&](int done) {
    const long long tb = t0 + (long long)done * C + urow;
    bf16* p = static_cast<bf16*>(a.out) + tb * ((long long)a.heads * a.dv) + (long long)head * a.dv + c0 + cu8;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      uint4 v;
      asm volatile("ld.shared.v4.b32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
                   : "r"(sQ + tile_off(urow + 32 * n, tid & 15)) : "memory");
      if (v_ok && tb + 32 * n < t1) *reinterpret_cast<uint4*>(p + (long long)(32 * n) * a.heads * a.dv) = v;
    }
  };

  // the rows that fetch() will read, on their way to the L2 while the current chunk is computed
  auto prefetch = [&](int chunk) {
    const long long tb = t0 + (long long)chunk * C + urow;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      if (tb + 32 * n < t1 && (tid & 7) == 0) {
        const bf16* pr = base + (tb + 32 * n) * a.stride;
        if (!STATE_ONLY && k_ok) asm volatile("prefetch.global.L2 [%0];" ::"l"(pr + a.off_q + head * a.dk + cu8));
        if (k_ok) asm volatile("prefetch.global.L2 [%0];" ::"l"(pr + a.off_k + head * a.dk + cu8));
        if (v_ok) asm volatile("prefetch.global.L2 [%0];" ::"l"(pr + a.off_v + head * a.dv + c0 + cu8));
      }
    }
  };

  bool ok = true;
  uint32_t phase = 0;
  fetch(0);
  int chunk = 0;
  for (; chunk < n_chunk; ++chunk, phase ^= 1u) {
    const int rows = min(C, n_tok - chunk * C);
    if (chunk + 1 < n_chunk) prefetch(chunk + 1);
    if (!STATE_ONLY && chunk > 0) store_out(chunk - 1);
    // ---- activated tiles, decayed keys, state -------------------------------------------------------
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int r = urow + 32 * n;
      const uint32_t off = tile_off(r, tid & 15);
      if (!STATE_ONLY) st_shared(sQ + off, silu8(rq[n]));
      const uint4 k = silu8(rk[n]);
      if (!STATE_ONLY) st_shared(sK + off, k);
      const float w = pw[max(rows - 1 - r, 0)];              // rows past the end are zero
      uint4 h, l;
      float2 f;
      f = unpack2(k.x); split2(f.x * w, f.y * w, h.x, l.x);
      f = unpack2(k.y); split2(f.x * w, f.y * w, h.y, l.y);
      f = unpack2(k.z); split2(f.x * w, f.y * w, h.z, l.z);
      f = unpack2(k.w); split2(f.x * w, f.y * w, h.w, l.w);
      st_shared(sKh + off, h);
      st_shared(sKl + off, l);
      st_shared(sV + off, silu8(rv[n]));
    }
    if (!STATE_ONLY) {
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
    if (warp == 0) {
      tc_fence_after();
      __syncwarp();
      const uint64_t qd = smem_desc(sQ, 16, 1024), kd = smem_desc(sK, 16, 1024);
      const uint64_t vd = smem_desc(sV, SLAB, 1024), khd = smem_desc(sKh, SLAB, 1024), kld = smem_desc(sKl, SLAB, 1024);
      const uint64_t shd = smem_desc(sSh, SLAB, 1024), sld = smem_desc(sSl, SLAB, 1024);
      if (!STATE_ONLY) {
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
      }
#pragma unroll
      for (int ks = 0; ks < 8; ++ks) {
        tc_mma_ss(tmem + 384u, khd + (uint64_t)(ks * 128), vd + (uint64_t)(ks * 128), IDESC_AB, ks > 0 ? 1u : 0u);
        tc_mma_ss(tmem + 384u, kld + (uint64_t)(ks * 128), vd + (uint64_t)(ks * 128), IDESC_AB, 1u);
      }
      tc_commit(bar_s);
    }
    if (!STATE_ONLY) {
      // ---- A -> P ------------------------------------------------------------------------------------
      ok = mbar_wait(bar_a, phase) && ok;
      tc_fence_after();
      float s[32];
      tc_ld32(tA, s);
      tc_wait_ld();
      tc_fence_before();
      __syncthreads();                                        // P is written over other warps' part of A
      tc_fence_after();
      const float* pr = pw + (row - cg * 32);                 // pr[-j]: weight of my column j (0 past my row)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        uint32_t ph[8], pl[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int j = h * 16 + 2 * i;
          const float x = s[j] * pr[-j], y = s[j + 1] * pr[-j - 1];
          split2(x, y, ph[i], pl[i]);
        }
        tc_st8(tP + h * 8u, ph);
        tc_st8(tP + 64u + h * 8u, pl);
      }
      tc_wait_st();
      tc_fence_before();
      __syncthreads();
      if (warp == 0) {
        tc_fence_after();
        __syncwarp();
        const uint64_t vd = smem_desc(sV, SLAB, 1024);
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {
          tc_mma_ts(tmem + 256u, tmem + (uint32_t)ks * 8u, vd + (uint64_t)(ks * 128), IDESC_B, ks > 0 ? 1u : 0u);
          tc_mma_ts(tmem + 256u, tmem + 64u + (uint32_t)ks * 8u, vd + (uint64_t)(ks * 128), IDESC_B, 1u);
        }
        tc_commit(bar_o);
      }
    }
    if (chunk + 1 < n_chunk) fetch(chunk + 1);
    // ---- state ---------------------------------------------------------------------------------------
    ok = mbar_wait(bar_s, phase) && ok;
    tc_fence_after();
    {
      const float dc = pw[rows];
      float t[32];
      tc_ld32(tS, t);
      tc_wait_ld();
#pragma unroll
      for (int i = 0; i < 32; ++i) S[i] = dc * S[i] + t[i];
    }
    // ---- output --------------------------------------------------------------------------------------
    if (!STATE_ONLY) {
      ok = mbar_wait(bar_o, phase) && ok;
      tc_fence_after();
      const float w = pw[min(row + 1, C)];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        float x[16], y[16];
        tc_ld16(tO1 + h * 16u, x);
        tc_ld16(tO2 + h * 16u, y);
        tc_wait_ld();
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          uint32_t p[4];
#pragma unroll
          for (int i = 0; i < 4; ++i)
            p[i] = pack_bf162(w * x[u * 8 + 2 * i] + y[u * 8 + 2 * i], w * x[u * 8 + 2 * i + 1] + y[u * 8 + 2 * i + 1]);
          st_shared(sQ + tile_off(row, cg * 4 + h * 2 + u), make_uint4(p[0], p[1], p[2], p[3]));   // Q is no longer read
        }
      }
    }
    if (__syncthreads_or(ok ? 0 : 1)) break;                  // a wait ran out somewhere in the CTA
  }
  if (chunk < n_chunk) {                                      // left early: wait (bounded) for what is still in flight
    if (tid == 0) atomicOr(a.status, kStatusWaitTimeout);
    if (!STATE_ONLY) {
      mbar_wait(bar_a, phase);
      mbar_wait(bar_o, phase);
    }
    mbar_wait(bar_s, phase);
  }
  if (!STATE_ONLY && chunk == n_chunk) store_out(n_chunk - 1);
  float* dst = STATE_ONLY ? segst : (last_seg ? cache : nullptr);
  if (dst != nullptr && row < a.dk) {
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
      const int c = c0 + cg * 32 + i;
      if (c < a.dv) *reinterpret_cast<float4*>(dst + (long long)row * a.dv + c) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    __syncwarp();
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
  }
}

}  // namespace

cudaError_t launch_lightning_tc5(const LightningArgs& a, cudaStream_t stream) {
  if (a.n_seq == 0) return cudaSuccess;
  const dim3 grid((unsigned)(a.n_seq * a.max_segs), (unsigned)a.heads, (unsigned)((a.dv + N - 1) / N));
  cudaError_t e;
  if (a.max_segs > 1) {
    e = cudaFuncSetAttribute(lightning_tc5_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (e != cudaSuccess) return e;
    lightning_tc5_kernel<true><<<grid, kThreads, kSmem, stream>>>(a);
    e = launch_lightning_segment_scan(a, stream);
    if (e != cudaSuccess) return e;
  }
  e = cudaFuncSetAttribute(lightning_tc5_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
  if (e != cudaSuccess) return e;
  lightning_tc5_kernel<false><<<grid, kThreads, kSmem, stream>>>(a);
  return cudaGetLastError();
}

}  // namespace hybrid
}  // namespace fa
