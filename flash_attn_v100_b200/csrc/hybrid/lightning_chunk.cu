// Decayed linear attention over prompts, chunk by chunk on the tensor cores (mma.sync, bfloat16 operands, fp32
// accumulators), sm_100a.
//
// With d the decay and S the state before a chunk of C = 64 tokens,
//     o_i = d^(i+1) S^T q_i + sum_{j <= i} d^(i-j) (q_i . k_j) v_j,      S <- d^C S + sum_j d^(C-1-j) k_j v_j^T.
// q, k, v are the activated projections, rounded to bfloat16 as every activation is.  Everything else that a product
// takes in - the state, the decayed scores, the decayed keys - is a fp32 number and enters as the sum of two bfloat16
// parts (high, low), i.e. with about 17 bits, so the recurrence keeps fp32 state and weights.
//
// CTA = (segment of a sequence, head, 64 value columns), eight warps.  For o each warp owns 16 rows x 32 columns; the
// state [DK, 64] stays in the warps' accumulators across the chunks, and its two parts are put into shared memory once per
// chunk for the S^T q product.  The next chunk's rows are fetched into registers while the current one is computed.
//
// Segments let few long sequences fill the GPU: a first launch computes what every segment adds to the state, a scan over
// the segments turns that into the state at the start of each, and the main launch then runs all segments side by side.
#include "../common.cuh"
#include "hybrid_common.cuh"
#include "lightning.cuh"

namespace fa {
namespace hybrid {
namespace {

constexpr int C = 64;          // tokens per chunk
constexpr int BV = 64;         // value columns per CTA
constexpr int kThreads = 256;

// Byte offset of 16-byte unit `u` of row `row` in a tile of 2^LOG units per row, swizzled for ldmatrix.
template <int UNITS>
__device__ __forceinline__ uint32_t tile_off(int row, int u) {
  return (uint32_t)((row * UNITS + (u ^ (row & 7))) * 16);
}

__device__ __forceinline__ float silu_fast(float z) {
  return __fdividef(z, 1.f + __expf(-z));      // both errors are far below the bfloat16 rounding that follows
}
__device__ __forceinline__ uint4 silu8(const uint4& raw) {
  union { uint4 u; __nv_bfloat162 h[4]; } a;
  a.u = raw;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    float2 f = __bfloat1622float2(a.h[i]);
    a.h[i] = __floats2bfloat162_rn(silu_fast(f.x), silu_fast(f.y));
  }
  return a.u;
}
// Two fp32 numbers as packed (high, low) bfloat16 parts.
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 r = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf162(x - r.x, y - r.y);
}
__device__ __forceinline__ float2 unpack2(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v)); }

template <int DK, bool STATE_ONLY>
__global__ void __launch_bounds__(kThreads, 2) lightning_chunk_kernel(const LightningArgs a) {
  constexpr int UK = DK / 8, UV = BV / 8;          // 16-byte units per row
  constexpr int NQ = C * UK / kThreads, NV = C * UV / kThreads;
  constexpr int MT = DK / 16;                      // 16-row blocks of the state
  constexpr int NS = MT;                           // its 8-column tiles per warp: 8 warps share MT x 8 tiles
  extern __shared__ __align__(1024) uint8_t sm[];
  const uint32_t sQ = smem_u32(sm), sK = sQ + C * DK * 2, sV = sK + C * DK * 2, sSh = sV + C * BV * 2, sSl = sSh + DK * BV * 2;
  float* pw = reinterpret_cast<float*>(sm + (2 * C * DK + C * BV + 2 * DK * BV) * 2);   // decay^0 .. decay^C
  const int seq = blockIdx.x / a.max_segs, seg = blockIdx.x - seq * a.max_segs;
  const int head = blockIdx.y, c0 = blockIdx.z * BV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;

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
  if (!slot_ok && tid == 0) atomicOr(a.status, 2);
  const long long hs = (long long)a.dk * a.dv;     // one head's state
  float* cache = slot_ok ? a.state + ((long long)slot * a.heads + head) * hs : nullptr;
  float* segst = a.max_segs > 1 ? a.seg_state + (((long long)seq * a.max_segs + seg) * a.heads + head) * hs : nullptr;
  const float d = a.decay[head];
  for (int i = tid; i <= C; i += kThreads) pw[i] = i == 0 ? 1.f : powf(d, (float)i);

  // ---- my part of the state: rows sr0 .. +15, columns sc0 .. +8 NS -------------------------------
  const int sr0 = (warp % MT) * 16, sc0 = (warp / MT) * NS * 8;
  float S[NS][4];
  const float* init = nullptr;
  if (!STATE_ONLY) {
    if (a.max_segs > 1) init = segst;
    else if (a.starts[seq] != 0) init = cache;
  }
#pragma unroll
  for (int n = 0; n < NS; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = sr0 + g + (e >> 1) * 8, c = c0 + sc0 + n * 8 + t4 * 2 + (e & 1);
      S[n][e] = (init != nullptr && r < a.dk && c < a.dv) ? init[(long long)r * a.dv + c] : 0.f;
    }
  auto put_state = [&]() {
#pragma unroll
    for (int n = 0; n < NS; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        uint32_t hi, lo;
        split2(S[n][2 * h], S[n][2 * h + 1], hi, lo);
        const int r = sr0 + g + h * 8, c = sc0 + n * 8 + t4 * 2;
        const uint32_t off = tile_off<UV>(r, c >> 3) + (uint32_t)(c & 7) * 2;
        asm volatile("st.shared.b32 [%0], %1;" ::"r"(sSh + off), "r"(hi) : "memory");
        asm volatile("st.shared.b32 [%0], %1;" ::"r"(sSl + off), "r"(lo) : "memory");
      }
  };

  // ---- fetching ---------------------------------------------------------------------------------
  const bf16* base = static_cast<const bf16*>(a.qkv);
  uint4 rq[STATE_ONLY ? 1 : NQ], rk[NQ], rv[NV];
  auto fetch = [&](int chunk) {
    const long long tb = t0 + (long long)chunk * C;
#pragma unroll
    for (int n = 0; n < NQ; ++n) {
      const int u = tid + n * kThreads, row = u / UK, cu = u % UK;
      const bool ok = tb + row < t1 && cu * 8 < a.dk;
      const bf16* p = base + (tb + row) * a.stride + head * a.dk + cu * 8;
      rk[n] = ok ? *reinterpret_cast<const uint4*>(p + a.off_k) : make_uint4(0, 0, 0, 0);
      if (!STATE_ONLY) rq[n] = ok ? *reinterpret_cast<const uint4*>(p + a.off_q) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int u = tid + n * kThreads, row = u / UV, cu = u % UV;
      const bool ok = tb + row < t1 && c0 + cu * 8 < a.dv;
      rv[n] = ok ? *reinterpret_cast<const uint4*>(base + (tb + row) * a.stride + a.off_v + head * a.dv + c0 + cu * 8)
                 : make_uint4(0, 0, 0, 0);
    }
  };
  auto st_shared = [](uint32_t addr, const uint4& v) {
    asm volatile("st.shared.v4.b32 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(v.x), "r"(v.y), "r"(v.z), "r"(v.w) : "memory");
  };
  auto put_rows = [&]() {
#pragma unroll
    for (int n = 0; n < NQ; ++n) {
      const int u = tid + n * kThreads, row = u / UK, cu = u % UK;
      st_shared(sK + tile_off<UK>(row, cu), silu8(rk[n]));
      if (!STATE_ONLY) st_shared(sQ + tile_off<UK>(row, cu), silu8(rq[n]));
    }
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int u = tid + n * kThreads, row = u / UV, cu = u % UV;
      st_shared(sV + tile_off<UV>(row, cu), silu8(rv[n]));
    }
  };

  // the warp's 16 output rows and 32 output columns; the rows of the warps of one scheduler add up to the same work
  const int orow = (warp < 4 ? warp >> 1 : 3 - ((warp - 4) >> 1)) * 16, ocol = (warp & 1) * 32;
  const int lrow = lane & 15, lhalf = lane >> 4;             // ldmatrix: row within 16, which 8-column half

  fetch(0);
  for (int chunk = 0; chunk < n_chunk; ++chunk) {
    __syncthreads();                                          // the previous chunk's tiles are no longer read
    put_rows();
    if (!STATE_ONLY) put_state();
    __syncthreads();
    if (chunk + 1 < n_chunk) fetch(chunk + 1);
    const int rows = min(C, n_tok - chunk * C);

    if (!STATE_ONLY) {
      uint32_t qf[MT][4];
#pragma unroll
      for (int k = 0; k < MT; ++k) ldmatrix_x4(qf[k], sQ + tile_off<UK>(orow + lrow, k * 2 + lhalf));
      float o[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
      // S^T q, high and low part of the state
#pragma unroll
      for (int k = 0; k < MT; ++k) {
#pragma unroll
        for (int n2 = 0; n2 < 2; ++n2) {
          const uint32_t off = tile_off<UV>(k * 16 + lrow, (ocol >> 3) + n2 * 2 + lhalf);
          uint32_t b[4];
          ldmatrix_x4_trans(b, sSh + off);
          mma_bf16_16816(o[n2 * 2], qf[k], b[0], b[1]);
          mma_bf16_16816(o[n2 * 2 + 1], qf[k], b[2], b[3]);
          ldmatrix_x4_trans(b, sSl + off);
          mma_bf16_16816(o[n2 * 2], qf[k], b[0], b[1]);
          mma_bf16_16816(o[n2 * 2 + 1], qf[k], b[2], b[3]);
        }
      }
      {
        const float w0 = pw[orow + g + 1], w1 = pw[orow + g + 9];
#pragma unroll
        for (int n = 0; n < 4; ++n) { o[n][0] *= w0; o[n][1] *= w0; o[n][2] *= w1; o[n][3] *= w1; }
      }
      // the chunk's own keys, 16 at a time
      for (int jb = 0; jb <= orow; jb += 16) {
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
        for (int k = 0; k < MT; ++k) {
          uint32_t b[4];
          // lanes 0-7: keys 0-7, first half; 8-15: second half; 16-31: keys 8-15 likewise
          ldmatrix_x4(b, sK + tile_off<UK>(jb + (lane & 7) + (lane >> 4) * 8, k * 2 + ((lane >> 3) & 1)));
          mma_bf16_16816(s[0], qf[k], b[0], b[1]);
          mma_bf16_16816(s[1], qf[k], b[2], b[3]);
        }
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int i = orow + g + h * 8, j = jb + n * 8 + t4 * 2;
            const float x = j <= i ? s[n][2 * h] * pw[i - j] : 0.f;
            const float y = j + 1 <= i ? s[n][2 * h + 1] * pw[i - j - 1] : 0.f;
            split2(x, y, ph[n * 2 + h], pl[n * 2 + h]);
          }
#pragma unroll
        for (int n2 = 0; n2 < 2; ++n2) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, sV + tile_off<UV>(jb + lrow, (ocol >> 3) + n2 * 2 + lhalf));
          mma_bf16_16816(o[n2 * 2], ph, b[0], b[1]);
          mma_bf16_16816(o[n2 * 2 + 1], ph, b[2], b[3]);
          mma_bf16_16816(o[n2 * 2], pl, b[0], b[1]);
          mma_bf16_16816(o[n2 * 2 + 1], pl, b[2], b[3]);
        }
      }
      bf16* out = static_cast<bf16*>(a.out) + (t0 + (long long)chunk * C) * ((long long)a.heads * a.dv) + (long long)head * a.dv + c0;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int i = orow + g + h * 8;
        if (i < rows) {
          bf16* orp = out + (long long)i * a.heads * a.dv;
#pragma unroll
          for (int n = 0; n < 4; ++n) {
            const int c = ocol + n * 8 + t4 * 2;
            if (c0 + c < a.dv) *reinterpret_cast<uint32_t*>(orp + c) = pack_bf162(o[n][2 * h], o[n][2 * h + 1]);
          }
        }
      }
    }

    // ---- state: S = d^rows S + sum_j (d^(rows-1-j) k_j) v_j^T ------------------------------------
    const float dc = pw[rows];
#pragma unroll
    for (int n = 0; n < NS; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[n][e] *= dc;
#pragma unroll
    for (int kb = 0; kb < C / 16; ++kb) {
      if (kb * 16 >= rows) break;
      uint32_t kf[4], kh[4], kl[4];
      // lanes 0-7: tokens 0-7, columns 0-7; 8-15: columns 8-15; 16-31: tokens 8-15 likewise
      ldmatrix_x4_trans(kf, sK + tile_off<UK>(kb * 16 + (lane & 7) + (lane >> 4) * 8, (sr0 >> 3) + ((lane >> 3) & 1)));
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int j = kb * 16 + (i >> 1) * 8 + t4 * 2;
        const float2 kk = unpack2(kf[i]);
        // rows past the end of the chunk are zero in the tile; their weight only has to be finite
        split2(kk.x * pw[max(rows - 1 - j, 0)], kk.y * pw[max(rows - 2 - j, 0)], kh[i], kl[i]);
      }
#pragma unroll
      for (int n2 = 0; n2 < NS / 2; ++n2) {
        uint32_t b[4];
        ldmatrix_x4_trans(b, sV + tile_off<UV>(kb * 16 + lrow, (sc0 >> 3) + n2 * 2 + lhalf));
        mma_bf16_16816(S[n2 * 2], kh, b[0], b[1]);
        mma_bf16_16816(S[n2 * 2 + 1], kh, b[2], b[3]);
        mma_bf16_16816(S[n2 * 2], kl, b[0], b[1]);
        mma_bf16_16816(S[n2 * 2 + 1], kl, b[2], b[3]);
      }
    }
  }
  float* dst = STATE_ONLY ? segst : (last_seg ? cache : nullptr);
  if (dst != nullptr) {
#pragma unroll
    for (int n = 0; n < NS; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = sr0 + g + (e >> 1) * 8, c = c0 + sc0 + n * 8 + t4 * 2 + (e & 1);
        if (r < a.dk && c < a.dv) dst[(long long)r * a.dv + c] = S[n][e];
      }
  }
}

// seg_state[seq, s] holds what segment s adds; turned in place into the state at the start of segment s.
__global__ void __launch_bounds__(256) lightning_segment_scan_kernel(const LightningArgs a) {
  const long long hs = (long long)a.dk * a.dv;
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  const int head = blockIdx.y, seq = blockIdx.z;
  if (i >= hs) return;
  long long n = a.cu[seq + 1] - (long long)a.cu[seq];
  const int n_seg = (int)((n + a.seg_len - 1) / a.seg_len);
  const int slot = a.slots[seq];
  float s = 0.f;
  if (a.starts[seq] != 0 && slot >= 0 && slot < a.n_slots) s = a.state[((long long)slot * a.heads + head) * hs + i];
  const float dl = powf(a.decay[head], (float)a.seg_len);
  float* p = a.seg_state + ((long long)seq * a.max_segs * a.heads + head) * hs + i;
  for (int k = 0; k < n_seg && k < a.max_segs; ++k, p += a.heads * hs) {
    const float add = k + 1 < n_seg ? *p : 0.f;     // the last segment's slot was not written
    *p = s;
    s = dl * s + add;
  }
}

constexpr int kBigChunk = 128, kBigCols = 128;     // lightning_tc5.cu

bool big_heads(int dk, int dv) { return dk > 64 || dv > 64; }

}  // namespace

cudaError_t launch_lightning_segment_scan(const LightningArgs& a, cudaStream_t stream) {
  lightning_segment_scan_kernel<<<dim3((unsigned)((a.dk * a.dv + 255) / 256), (unsigned)a.heads, (unsigned)a.n_seq), 256, 0, stream>>>(a);
  return cudaGetLastError();
}

int lightning_segments(int n_seq, int heads, int dk, int dv, int max_len, int sm_count, int* seg_len) {
  // as many CTAs as run side by side (one per SM of the tcgen05 kernel, two of the other), in segments of at least 512
  // tokens: a segment's keys and values are read twice, which only pays while SMs would stay empty
  const bool big = big_heads(dk, dv);
  const int chunk = big ? kBigChunk : C, slots = (big ? 1 : 2) * sm_count;
  const long long tasks = (long long)n_seq * heads * ((dv + (big ? kBigCols : BV) - 1) / (big ? kBigCols : BV));
  const long long segs = tasks * 2 > slots ? 1 : slots / tasks;
  long long len = (max_len + segs - 1) / segs;
  if (len < 512) len = 512;
  len = (len + chunk - 1) / chunk * chunk;
  *seg_len = (int)len;
  return (int)((max_len + len - 1) / len);
}

bool lightning_chunk_supported(const LightningArgs& a) {
  return a.cu != nullptr && a.dk <= 128 && a.dk % 8 == 0 && a.dv % 8 == 0 && a.stride % 8 == 0 && a.off_q % 8 == 0 && a.off_k % 8 == 0 &&
         a.off_v % 8 == 0 && (reinterpret_cast<uintptr_t>(a.qkv) & 15) == 0 && (reinterpret_cast<uintptr_t>(a.out) & 15) == 0;
}

cudaError_t launch_lightning_chunk(const LightningArgs& a, cudaStream_t stream) {
  if (a.n_seq == 0) return cudaSuccess;
  if (big_heads(a.dk, a.dv)) return launch_lightning_tc5(a, stream);
  constexpr int DK = 64;
  constexpr int smem = (2 * C * DK + C * BV + 2 * DK * BV) * 2 + (C + 1) * 4;
  const dim3 grid((unsigned)(a.n_seq * a.max_segs), (unsigned)a.heads, (unsigned)((a.dv + BV - 1) / BV));
  cudaError_t e;
  if (a.max_segs > 1) {
    e = cudaFuncSetAttribute(lightning_chunk_kernel<DK, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    lightning_chunk_kernel<DK, true><<<grid, kThreads, smem, stream>>>(a);
    e = launch_lightning_segment_scan(a, stream);
    if (e != cudaSuccess) return e;
  }
  e = cudaFuncSetAttribute(lightning_chunk_kernel<DK, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  lightning_chunk_kernel<DK, false><<<grid, kThreads, smem, stream>>>(a);
  return cudaGetLastError();
}

}  // namespace hybrid
}  // namespace fa
