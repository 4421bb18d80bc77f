// Attention in the latent space on the tensor cores (mma.sync, bfloat16 operands, fp32 scores, weights' sums and
// accumulators), sm_100a: decode steps and short portions of prompts.
//
// All heads read the same cached rows, so a key tile (64 tokens) is fetched once and serves every head of the block (16 or
// 32, the M rows of the MMAs) as key and as value.  The (row, key tile) units of the batch are numbered row by row and cut
// into equal runs, one per CTA, whatever the lengths; a row that is cut leaves partial sums that a second kernel merges.
//
// Sixteen warps compute.  Scores: warp = (a quarter of the tile's keys) x (one 16-column step of every slab); the four partial
// score tiles are added up in shared memory by the softmax.  Values: warp = 8 columns of every other slab.  (With these shares
// every shared-memory address is a per-warp base plus a constant.)  A seventeenth warp fetches the tiles by TMA, one box of 16
// rows x 64 columns per page and slab (128-byte swizzle), one tile ahead.  Waits are bounded; one that runs out sets the status
// word.
#include <math_constants.h>

#include "../common.cuh"
#include "hybrid_common.cuh"
#include "latent_attention.cuh"

namespace fa {
namespace hybrid {
namespace {

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion,
                                  CUtensorMapFloatOOBfill);

constexpr int KT = 64;         // keys per tile
constexpr int kCompute = 512;  // threads that compute
constexpr int kThreads = kCompute + 32;
constexpr int kWarps = kThreads / 32;
constexpr int kSPad = KT + 8;  // row stride of the partial score tiles
constexpr int kSlab = KT * 128;

// Unit (16 bytes) `u` of key `key`: 128-byte-swizzled slabs of 64 columns.
__device__ __forceinline__ uint32_t key_off(int key, int u) {
  return (uint32_t)((u >> 3) * kSlab + key * 128 + ((u ^ key) & 7) * 16);
}
// Unit `u` of query row `row`, rows of UNITS units.
template <int UNITS>
__device__ __forceinline__ uint32_t q_off(int row, int u) {
  return (uint32_t)((row * UNITS + ((u & ~7) | ((u ^ row) & 7))) * 16);
}

__device__ __forceinline__ int row_tiles_of(const LatentAttentionArgs& a, long long row) {
  const int n = a.positions[row] + 1;
  return n > 0 ? (n + KT - 1) / KT : 1;
}

// Inclusive scan over the block of one int per thread; `buf` holds one int per warp.
__device__ __forceinline__ int block_scan(int v, int* buf) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int t = __shfl_up_sync(0xffffffffu, v, o);
    if (lane >= o) v += t;
  }
  if (lane == 31) buf[warp] = v;
  __syncthreads();
  int add = 0;
  for (int i = 0; i < warp; ++i) add += buf[i];
  __syncthreads();
  return v + add;
}

// KS: slabs of 64 columns = 16-column steps per warp quarter (4 * 16 * KS >= kv_rank + rot_dim); MB: 16-head blocks.
template <int KS, int MB>
__global__ void __launch_bounds__(kThreads, 1) latent_decode_kernel(const __grid_constant__ CUtensorMap pool_map,
                                                                    const LatentAttentionArgs a) {
  constexpr int UNITS = KS * 8;                    // 16-byte units per key row
  constexpr int STAGE = KS * kSlab;
  constexpr int M = 16 * MB;
  constexpr int SBYTES = 4 * M * kSPad * 4, QBYTES = M * UNITS * 16;
  constexpr int TPR = 16;                          // softmax threads per row, four keys each
  constexpr int NT = (KS + 1) / 2;                 // 8-column value tiles per warp
  extern __shared__ uint8_t sm_dyn[];
  uint8_t* sm = sm_dyn + ((1024u - (smem_u32(sm_dyn) & 1023u)) & 1023u);
  const uint32_t sKV = smem_u32(sm);
  float* sS = reinterpret_cast<float*>(sm + 2 * STAGE);            // [4][M][kSPad]
  const uint32_t sQ = smem_u32(sS) + SBYTES;                       // [M][UNITS] units: the current row's queries
  const uint32_t sP = sQ + QBYTES;                                 // [M][KT] bfloat16, swizzled
  float* sAlpha = reinterpret_cast<float*>(sm + 2 * STAGE + SBYTES + QBYTES + M * KT * 2);   // [M]
  float* sL = sAlpha + M;                                          // [M]
  int* scan_buf = reinterpret_cast<int*>(sL + M);                  // [kWarps]
  int* found = scan_buf + kWarps;                                  // [2] first row, its first unit
  const uint32_t bars = smem_u32(scan_buf + kWarps + 3);           // [2] tile has landed, [2] tile is no longer read
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int cta = blockIdx.x, h0 = blockIdx.y * M;
  const int R = a.kv_rank, D = R + a.rot_dim;

  // ---- my run of units --------------------------------------------------------------------------
  int total = 0, mine = 0, upto = 0;               // of my row in the last block of rows: its tiles, tiles up to and with it
  for (long long r0 = 0; r0 < a.rows; r0 += kThreads) {
    mine = r0 + tid < a.rows ? row_tiles_of(a, r0 + tid) : 0;
    upto = total + block_scan(mine, scan_buf);
    if (cta == 0 && blockIdx.y == 0 && r0 + tid < a.rows) a.row_tiles[r0 + tid + 1] = upto;
    if (tid == kThreads - 1) found[0] = upto;
    __syncthreads();
    total = found[0];
    __syncthreads();
  }
  if (cta == 0 && blockIdx.y == 0 && tid == 0) a.row_tiles[0] = 0;
  const int per = (total + a.n_cta - 1) / a.n_cta;
  const int u0 = cta * per, u1 = min(u0 + per, total);
  if (u0 >= u1) return;
  if (a.rows <= kThreads) {
    if (mine > 0 && upto - mine <= u0 && u0 < upto) { found[0] = tid; found[1] = upto - mine; }
    __syncthreads();
  } else {
    int base = 0;
    for (long long r0 = 0; r0 < a.rows; r0 += kThreads) {
      const int v = r0 + tid < a.rows ? row_tiles_of(a, r0 + tid) : 0;
      const int inc = base + block_scan(v, scan_buf);
      if (v > 0 && inc - v <= u0 && u0 < inc) { found[0] = (int)(r0 + tid); found[1] = inc - v; }
      if (tid == kThreads - 1) scan_buf[0] = inc;
      __syncthreads();
      base = scan_buf[0];
      __syncthreads();
      if (base > u0) break;
    }
  }
  const int first_row = found[0];
  if (tid == 0) {
    mbar_init(bars, 4 * KS);                        // one arrival per box
    mbar_init(bars + 8, 4 * KS);
    mbar_init(bars + 16, kCompute / 32);            // one arrival per computing warp
    mbar_init(bars + 24, kCompute / 32);
    mbar_fence_init();
    fence_proxy_async();
    tma_prefetch_desc(&pool_map);
  }
  __syncthreads();
  struct Cursor { int row, tile, tiles, n; };
  auto start_row = [&](Cursor& c, int row) { c.row = row; c.tile = 0; c.n = a.positions[row] + 1; c.tiles = c.n > 0 ? (c.n + KT - 1) / KT : 1; };
  auto advance = [&](Cursor& c) {
    if (++c.tile == c.tiles && c.row + 1 < a.rows) start_row(c, c.row + 1);
  };

  bool late = false;
  auto wait = [&](uint32_t bar, uint32_t parity) {
    if (!late) late = !mbar_wait(bar, parity);
  };

  if (warp == kCompute / 32) {
    // ---- copies: lane l fetches boxes l and l + 32 of every tile ------------------------------------
    constexpr int NB = (4 * KS + 31) / 32;
    bool bad = false;
    // page of the cursor's tile that a box comes from, checked when it is used; keys past the end: the tile's first page (any
    // finite rows will do, their weights are zero)
    auto box_page = [&](const Cursor& c, int box) {
      const int seq = a.tok_seq[c.row];
      int blk = c.tile * (KT / 16) + box / KS;
      if (blk * 16 >= c.n) blk = c.tile * (KT / 16);
      return seq >= 0 && seq < a.n_seq && c.n > 0 && blk < a.max_blocks ? a.block_table[(long long)seq * a.max_blocks + blk] : -1;
    };
    Cursor nxt;
    start_row(nxt, first_row);
    nxt.tile = u0 - found[1];
    int page[NB];
#pragma unroll
    for (int i = 0; i < NB; ++i) page[i] = lane + 32 * i < 4 * KS ? box_page(nxt, lane + 32 * i) : 0;
#pragma unroll 1
    for (int u = u0; u < u1; ++u) {
      const int k = u - u0, stage = k & 1;
      if (k >= 2) wait(bars + 16 + 8 * stage, (uint32_t)((k >> 1) - 1) & 1u);
#pragma unroll
      for (int i = 0; i < NB; ++i) {
        const int box = lane + 32 * i;
        if (box < 4 * KS) {
          if (page[i] < 0 || page[i] >= a.n_blocks) { bad = true; page[i] = 0; }
          mbar_expect_tx(bars + 8 * stage, 2048);
          tma_load_2d_nohint(sKV + stage * STAGE + (box % KS) * kSlab + (box / KS) * 2048, &pool_map, (box % KS) * 64, page[i] * 16,
                             bars + 8 * stage);
        }
      }
      if (u + 1 < u1) {
        advance(nxt);
#pragma unroll
        for (int i = 0; i < NB; ++i)
          if (lane + 32 * i < 4 * KS) page[i] = box_page(nxt, lane + 32 * i);
      }
    }
    // leave only when every copy has landed
    for (int k = u1 - u0 >= 2 ? u1 - u0 - 2 : 0; k < u1 - u0; ++k)
      if (!mbar_wait(bars + 8 * (k & 1), (uint32_t)(k >> 1) & 1u)) late = true;
    if (bad) atomicOr(a.status, kStatusBadPageId);
    if (late) atomicOr(a.status, kStatusWaitTimeout);
    return;
  }
  auto sync = [&]() { asm volatile("bar.sync 1, %0;" ::"n"(kCompute) : "memory"); };

  // ---- per-row state ----------------------------------------------------------------------------
  const int slice = warp & 3, kquarter = warp >> 2;
  // my lane's ldmatrix addresses within a stage (scores: my 16 keys; values: all keys; queries: 16 heads)
  const uint32_t k_base = key_off(kquarter * 16 + (lane & 7) + (lane >> 4) * 8, slice * 2 + ((lane >> 3) & 1)), v_base = key_off(lane, warp);
  const uint32_t q_base = sQ + q_off<UNITS>(lane & 15, slice * 2 + (lane >> 4));
  float o[MB][NT][4];
  // All threads; a barrier follows before the queries are read.
  auto load_q = [&](long long row) {
    const int half = a.rot_dim / 2;
#pragma unroll 1
    for (int idx = tid; idx < M * UNITS; idx += kCompute) {
      const int m = idx / UNITS, u = idx - m * UNITS, c = u * 8, head = h0 + m;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (head < a.heads) {
        if (c < R) {
          v = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(a.q_abs) + (row * a.heads + head) * R + c);
        } else if (c < D) {
          const bf16* qr = static_cast<const bf16*>(a.q) + (row * a.heads + head) * a.q_stride + a.q_off;
          float e[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            const int i = c - R + j, f = i < half ? i : i - half;
            const float cs = a.cos_t[row * half + f], sn = a.sin_t[row * half + f];
            e[j] = i < half ? to_f(qr[i]) * cs - to_f(qr[i + half]) * sn : to_f(qr[i]) * cs + to_f(qr[i - half]) * sn;
          }
          v = make_uint4(pack_bf162(e[0], e[1]), pack_bf162(e[2], e[3]), pack_bf162(e[4], e[5]), pack_bf162(e[6], e[7]));
        }
      }
      asm volatile("st.shared.v4.b32 [%0], {%1,%2,%3,%4};" ::"r"(sQ + q_off<UNITS>(m, u)), "r"(v.x), "r"(v.y), "r"(v.z), "r"(v.w) : "memory");
    }
#pragma unroll
    for (int m = 0; m < MB; ++m)
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[m][n][e] = 0.f;
  };
  const int srow = tid / TPR, sk0 = (tid % TPR) * 4;         // softmax: my head row and its four keys
  float m_run = -CUDART_INF_F, l_run = 0.f;
  const float sc = a.scale * 1.4426950408889634f;

  Cursor cur;
  start_row(cur, first_row);
  cur.tile = u0 - found[1];
  int piece_tile0 = cur.tile;
  load_q(cur.row);
  sync();

#pragma unroll 1
  for (int u = u0; u < u1; ++u) {
    const int stage = (u - u0) & 1;
    wait(bars + 8 * stage, (uint32_t)((u - u0) >> 1) & 1u);
    // ---- partial scores -------------------------------------------------------------------------
    {
      float s[MB][2][4];
#pragma unroll
      for (int m = 0; m < MB; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[m][n][e] = 0.f;
      const uint32_t kb = sKV + stage * STAGE + k_base;
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        uint32_t b[4];
        ldmatrix_x4(b, kb + k * kSlab);
#pragma unroll
        for (int m = 0; m < MB; ++m) {
          uint32_t q[4];
          ldmatrix_x4(q, q_base + (uint32_t)(m * 16 * UNITS * 16 + k * 128));
          mma_bf16_16816(s[m][0], q, b[0], b[1]);
          mma_bf16_16816(s[m][1], q, b[2], b[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < MB; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int h = 0; h < 2; ++h)
            *reinterpret_cast<float2*>(sS + (slice * M + m * 16 + g + h * 8) * kSPad + kquarter * 16 + n * 8 + t4 * 2) =
                make_float2(s[m][n][2 * h], s[m][n][2 * h + 1]);
    }
    sync();
    // ---- softmax of my row's keys ---------------------------------------------------------------
    if (srow < M) {                                 // (whole warps)
      const int valid = cur.n - cur.tile * KT - sk0;
      float4 v = *reinterpret_cast<const float4*>(sS + srow * kSPad + sk0);
#pragma unroll
      for (int q = 1; q < 4; ++q) {
        const float4 w = *reinterpret_cast<const float4*>(sS + (q * M + srow) * kSPad + sk0);
        v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
      }
      v.x = valid > 0 ? v.x * sc : -CUDART_INF_F;
      v.y = valid > 1 ? v.y * sc : -CUDART_INF_F;
      v.z = valid > 2 ? v.z * sc : -CUDART_INF_F;
      v.w = valid > 3 ? v.w * sc : -CUDART_INF_F;
      float mx = fmaxf(fmaxf(v.x, v.y), fmaxf(v.z, v.w));
#pragma unroll
      for (int w = 1; w < TPR; w <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
      const float m_new = fmaxf(m_run, mx);
      const float ref = m_new == -CUDART_INF_F ? 0.f : m_new;
      const float alpha = fast_exp2(m_run - ref);   // 0 at the row's first tile
      v.x = fast_exp2(v.x - ref); v.y = fast_exp2(v.y - ref); v.z = fast_exp2(v.z - ref); v.w = fast_exp2(v.w - ref);
      float sum = (v.x + v.y) + (v.z + v.w);
#pragma unroll
      for (int w = 1; w < TPR; w <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
      l_run = l_run * alpha + sum;
      m_run = m_new;
      const uint32_t addr = sP + (uint32_t)((srow * 8 + ((sk0 >> 3) ^ (srow & 7))) * 16 + (sk0 & 7) * 2);
      asm volatile("st.shared.v2.b32 [%0], {%1,%2};" ::"r"(addr), "r"(pack_bf162(v.x, v.y)), "r"(pack_bf162(v.z, v.w)) : "memory");
      if (tid % TPR == 0) { sAlpha[srow] = alpha; sL[srow] = l_run; }
    }
    sync();
    // ---- values: my columns of the latents --------------------------------------------------------
    {
#pragma unroll
      for (int m = 0; m < MB; ++m) {
        const float a0 = sAlpha[m * 16 + g], a1 = sAlpha[m * 16 + g + 8];
        if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
          for (int n = 0; n < NT; ++n) { o[m][n][0] *= a0; o[m][n][1] *= a0; o[m][n][2] *= a1; o[m][n][3] *= a1; }
        }
      }
#pragma unroll
      for (int k2 = 0; k2 < KT / 32; ++k2) {        // 32 keys at a time
        uint32_t pf[MB][2][4];
#pragma unroll
        for (int m = 0; m < MB; ++m)
#pragma unroll
          for (int k = 0; k < 2; ++k) {
            const int r = m * 16 + (lane & 15), c8 = (k2 * 2 + k) * 2 + (lane >> 4);
            ldmatrix_x4(pf[m][k], sP + (uint32_t)((r * 8 + (c8 ^ (r & 7))) * 16));
          }
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          if ((n * 16 + warp) * 8 < R) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, sKV + stage * STAGE + v_base + n * 2 * kSlab + k2 * 32 * 128);
#pragma unroll
            for (int m = 0; m < MB; ++m) {
              mma_bf16_16816(o[m][n], pf[m][0], b[0], b[1]);
              mma_bf16_16816(o[m][n], pf[m][1], b[2], b[3]);
            }
          }
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(bars + 16 + 8 * stage);
    // ---- end of a row or of my run ------------------------------------------------------------------
    const bool row_end = cur.tile + 1 == cur.tiles;
    if (row_end || u + 1 == u1) {
      const bool whole = row_end && piece_tile0 == 0;
      const int which = cur.row == first_row ? 0 : 1;
      if (!whole && tid % TPR == 0 && srow < M && h0 + srow < a.heads) {
        float* ml = a.part_ml + (((long long)cta * 2 + which) * a.heads + h0 + srow) * 2;
        ml[0] = m_run;
        ml[1] = l_run;
      }
#pragma unroll
      for (int m = 0; m < MB; ++m)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int head = h0 + m * 16 + g + h * 8;
          if (head < a.heads) {
            float f = 1.f;
            if (whole) {
              const float l = sL[m * 16 + g + h * 8];
              f = l > 0.f ? 1.f / l : 0.f;
              if (a.gate != nullptr) f *= sigmoid_f(to_f(static_cast<const bf16*>(a.gate)[(long long)cur.row * a.gate_stride + head]));
            }
#pragma unroll
            for (int n = 0; n < NT; ++n) {
              const int c = (n * 16 + warp) * 8 + t4 * 2;
              if (c < R) {
                const float x = o[m][n][2 * h] * f, y = o[m][n][2 * h + 1] * f;
                if (whole)
                  *reinterpret_cast<uint32_t*>(static_cast<bf16*>(a.out) + ((long long)cur.row * a.heads + head) * R + c) = pack_bf162(x, y);
                else
                  *reinterpret_cast<float2*>(a.part_o + (((long long)cta * 2 + which) * a.heads + head) * R + c) = make_float2(x, y);
              }
            }
          }
        }
      if (u + 1 < u1) {
        m_run = -CUDART_INF_F;
        l_run = 0.f;
        load_q(cur.row + 1);
        sync();
        piece_tile0 = 0;
      }
    }
    if (u + 1 < u1) advance(cur);
  }
  if (late && lane == 0) atomicOr(a.status, kStatusWaitTimeout);
}

// Rows that several CTAs worked on: log-sum-exp merge of their partial sums.  One CTA per (row, head).
constexpr int kMergeThreads = 128;
__global__ void __launch_bounds__(kMergeThreads) latent_decode_merge_kernel(const LatentAttentionArgs a) {
  extern __shared__ float weight[];                 // [pieces of the row] (n_cta at most)
  __shared__ float red[2 * kMergeThreads / 32];
  const long long row = blockIdx.x;
  const int head = blockIdx.y, tid = threadIdx.x;
  const int b0 = a.row_tiles[row], b1 = a.row_tiles[row + 1], total = a.row_tiles[a.rows];
  const int per = (total + a.n_cta - 1) / a.n_cta;
  const int c0 = b0 / per, n = (b1 - 1) / per - c0 + 1;
  if (n == 1) return;                               // one CTA had the whole row
  // the row is a CTA's first one exactly if the CTA's run starts inside it or at its first unit
  auto piece = [&](int i) { return ((long long)(c0 + i) * 2 + ((c0 + i) * per >= b0 ? 0 : 1)) * a.heads + head; };
  float m = -CUDART_INF_F;
  for (int i = tid; i < n; i += kMergeThreads) m = fmaxf(m, a.part_ml[piece(i) * 2]);
  m = warp_max(m);
  if ((tid & 31) == 0) red[tid >> 5] = m;
  __syncthreads();
  m = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
  float l = 0.f;
  for (int i = tid; i < n; i += kMergeThreads) {
    const float w = exp2f(a.part_ml[piece(i) * 2] - m);
    weight[i] = w;
    l += w * a.part_ml[piece(i) * 2 + 1];
  }
  l = block_sum(l, red + 4);
  float f = l > 0.f ? 1.f / l : 0.f;
  if (a.gate != nullptr) f *= sigmoid_f(to_f(static_cast<const bf16*>(a.gate)[row * a.gate_stride + head]));
  bf16* out = static_cast<bf16*>(a.out) + (row * a.heads + head) * a.kv_rank;
  for (int i = tid * 4; i < a.kv_rank; i += kMergeThreads * 4) {
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
    for (int c = 0; c < n; ++c) {
      float v[4];
      load_n<4>(a.part_o + piece(c) * a.kv_rank + i, v);
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[j] += weight[c] * v[j];
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[j] *= f;
    store_n<4>(out + i, acc);
  }
}

template <int KS, int MB>
cudaError_t launch_t(const LatentAttentionArgs& a, const CUtensorMap& map, cudaStream_t s) {
  constexpr int M = 16 * MB;
  constexpr int smem = 1024 + 2 * KS * kSlab + 4 * M * kSPad * 4 + M * KS * 128 + M * KT * 2 + 2 * M * 4 + (kWarps + 3) * 4 + 4 * 8;
  static_assert(smem <= 227 * 1024, "shared memory plan exceeds the SM");
  cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<KS, MB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  latent_decode_kernel<KS, MB><<<dim3((unsigned)a.n_cta, (unsigned)((a.heads + M - 1) / M)), kThreads, smem, s>>>(map, a);
  latent_decode_merge_kernel<<<dim3((unsigned)a.rows, (unsigned)a.heads), kMergeThreads, a.n_cta * sizeof(float), s>>>(a);
  return cudaGetLastError();
}

int ks_of(int D) { return D <= 128 ? 2 : (D <= 192 ? 3 : (D <= 320 ? 5 : 9)); }

}  // namespace

bool latent_decode_supported(const LatentAttentionArgs& a) {
  return a.kv_rank % 8 == 0 && a.rot_dim % 8 == 0 && a.rot_dim > 0 && a.kv_rank + a.rot_dim <= 576 && a.pool_stride % 8 == 0 &&
         a.rows < (1ll << 30) && (reinterpret_cast<uintptr_t>(a.pool) & 15) == 0 && (reinterpret_cast<uintptr_t>(a.q_abs) & 15) == 0 &&
         (reinterpret_cast<uintptr_t>(a.out) & 15) == 0;
}

int latent_decode_ctas(int heads, int sm_count) {
  const int blocks = heads <= 16 ? 1 : (heads + 31) / 32;
  const int n = sm_count / blocks;
  return n > 0 ? n : 1;
}

cudaError_t launch_latent_decode(const LatentAttentionArgs& a, void* encode_fn, cudaStream_t s) {
  if (a.rows == 0) return cudaSuccess;
  CUtensorMap map;
  const cuuint64_t dims[2] = {(cuuint64_t)a.pool_stride, (cuuint64_t)a.n_blocks * 16};
  const cuuint64_t strides[1] = {(cuuint64_t)a.pool_stride * 2};
  const cuuint32_t box[2] = {64, 16}, estr[2] = {1, 1};
  if (reinterpret_cast<EncodeTiledFn>(encode_fn)(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(a.pool), dims, strides, box, estr,
                                                 CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                                                 CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return cudaErrorInvalidValue;
  const int ks = ks_of(a.kv_rank + a.rot_dim);
  if (a.heads <= 16) {
    if (ks == 2) return launch_t<2, 1>(a, map, s);
    if (ks == 3) return launch_t<3, 1>(a, map, s);
    if (ks == 5) return launch_t<5, 1>(a, map, s);
    return launch_t<9, 1>(a, map, s);
  }
  if (ks == 2) return launch_t<2, 2>(a, map, s);
  if (ks == 3) return launch_t<3, 2>(a, map, s);
  if (ks == 5) return launch_t<5, 2>(a, map, s);
  return launch_t<9, 2>(a, map, s);
}

}  // namespace hybrid
}  // namespace fa
