// Grouped-query attention of single query rows on paged keys and values inside chunks (decode steps, short portions), bfloat16,
// sm_100a.
//
// CTA = (query row, KV head and block of up to 16 query heads, range of the row's keys), four warps, two CTAs per SM.  A warp streams
// its own pages (page i of the range goes to warp i mod 4) through a private ring of shared-memory stages filled by cp.async, so there
// is no barrier until the warps' results are merged; the query heads of a KV head are the rows of the MMAs, so every key and value is
// read from memory once.  S = Q K^T and O += P V run on mma.sync m16n8k16 with fp32 accumulators; the softmax is fp32, base 2,
// online; the distance bias is added to the fp32 scores.  Rows whose keys are shared by several CTAs are merged by a second kernel,
// otherwise the gate is applied and the row written here.
#include <math_constants.h>

#include "../common.cuh"
#include "../hybrid/hybrid_common.cuh"
#include "kv_attention.cuh"

namespace fa {
namespace mixers {

using hybrid::bf16;
using hybrid::sigmoid_f;
using hybrid::to_f;

namespace {

constexpr int kWarps = 4;
constexpr int kThreads = kWarps * 32;
constexpr float kLog2e = 1.4426950408889634f;

// Byte offset of 16-byte unit `u` of row `row` in a page of COLS columns, swizzled for ldmatrix.
template <int COLS>
__device__ __forceinline__ uint32_t page_off(int row, int u) {
  return (uint32_t)(row * COLS * 2 + ((u ^ (row & 7)) & (COLS / 8 - 1)) * 16);
}

template <int KD, int VD>
struct Plan {
  static constexpr int STAGE = 16 * (KD + VD) * 2;
  static constexpr int STAGES = 24576 / STAGE;
  static constexpr int RING = kWarps * STAGES * STAGE;
  static constexpr int MERGE = kWarps * 16 * (VD + 2) * 4;
  static constexpr int BYTES = RING > MERGE ? RING : MERGE;
};

// KD, VD: columns of keys and values, padded with zeros; HM: at most 8 query heads per KV head (rows 8 to 15 of the MMAs are unused).
template <int KD, int VD, bool HM>
__global__ void __launch_bounds__(kThreads, 2) kv_decode_kernel(const KvAttentionArgs a, const int head_blocks) {
  using P = Plan<KD, VD>;
  constexpr int KS = KD / 16, NT = VD / 8;
  extern __shared__ __align__(128) uint8_t smem[];
  const long long row = blockIdx.x / a.splits;
  const int split = (int)(blockIdx.x - row * a.splits);
  const int kvh = blockIdx.y / head_blocks, hb = blockIdx.y - kvh * head_blocks;
  const int rep = a.heads / a.kv_heads;
  const int h0 = kvh * rep + hb * 16, nh = min(16, rep - hb * 16);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int seq = a.pg.tok_seq[row], pos = a.pg.positions[row];
  const bool bad = seq < 0 || seq >= a.pg.n_seq || pos < 0 || (pos >> 4) >= a.pg.max_blocks;
  if (bad && tid == 0) atomicOr(a.status, kStatusBadPageId);
  const int first = a.chunk > 0 ? pos - pos % a.chunk : 0;
  // this CTA's pages [p0, p1)
  int p0 = first >> 4, p1 = bad ? p0 : (pos >> 4) + 1;
  {
    const int per = (p1 - p0 + a.splits - 1) / a.splits;
    p0 += split * per;
    if (p1 > p0 + per) p1 = p0 + per;
  }
  const int n_mine = p1 > p0 + warp ? (p1 - p0 - warp + kWarps - 1) / kWarps : 0;     // my pages: p0 + warp + i kWarps

  const uint32_t ring = smem_u32(smem) + (uint32_t)(warp * P::STAGES * P::STAGE);
  const int32_t* table = a.pg.block_table + (long long)(bad ? 0 : seq) * a.pg.max_blocks;
  const bf16* kp = static_cast<const bf16*>(a.k_pool);
  const bf16* vp = static_cast<const bf16*>(a.v_pool);
  int ids = -1;                // the lane's entry of the next 32 pages' numbers
  auto fetch = [&](int i) {
    if ((i & 31) == 0) {
      const int p = p0 + warp + (i + lane) * kWarps;
      ids = i + lane < n_mine ? table[p] : 0;
      if (ids < 0 || ids >= a.pg.n_blocks) {
        atomicOr(a.status, kStatusBadPageId);
        ids = -1;
      }
    }
    const int page = __shfl_sync(0xffffffffu, ids, i & 31);
    const uint32_t st = ring + (uint32_t)((i % P::STAGES) * P::STAGE);
    const long long at = (long long)(page < 0 ? 0 : page) * a.kv_heads + kvh;
    const bf16 *k = kp + at * 16 * a.dim, *v = vp + at * 16 * a.vdim;
#pragma unroll
    for (int n = 0; n < KD / 16; ++n) {
      const int u = lane + n * 32, r = u / (KD / 8), c = u % (KD / 8);
      const bool ok = page >= 0 && c * 8 < a.dim;
      cp_async_16(st + page_off<KD>(r, c), ok ? k + r * a.dim + c * 8 : kp, ok);
    }
#pragma unroll
    for (int n = 0; n < VD / 16; ++n) {
      const int u = lane + n * 32, r = u / (VD / 8), c = u % (VD / 8);
      const bool ok = page >= 0 && c * 8 < a.vdim;
      cp_async_16(st + 16 * KD * 2 + page_off<VD>(r, c), ok ? v + r * a.vdim + c * 8 : vp, ok);
    }
  };
#pragma unroll
  for (int i = 0; i < P::STAGES - 1; ++i) {
    if (i < n_mine) fetch(i);
    cp_async_commit();
  }

  // ---- queries: the MMAs' rows are heads ------------------------------------------------------------
  uint32_t q[KS][4];
  const bf16* qr = static_cast<const bf16*>(a.q) + (row * a.heads + h0) * a.dim;
#pragma unroll
  for (int k = 0; k < KS; ++k)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = g + (e & 1) * 8, c = k * 16 + (e >> 1) * 8 + t4 * 2;
      q[k][e] = (!HM || (e & 1) == 0) && h < nh && c < a.dim ? *reinterpret_cast<const uint32_t*>(qr + (long long)h * a.dim + c) : 0u;
    }
  const float sc = a.scale * kLog2e;
  float slope[2] = {0.f, 0.f};
#pragma unroll
  for (int h = 0; h < 2; ++h)
    if (a.slopes != nullptr && g + h * 8 < nh) slope[h] = a.slopes[h0 + g + h * 8] * kLog2e;

  constexpr int HR = HM ? 1 : 2;     // rows per thread
  float o[NT][4];
  float m[2] = {-CUDART_INF_F, -CUDART_INF_F}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;

  const int lrow = lane & 15, lhalf = lane >> 4;
  for (int i = 0; i < n_mine; ++i) {
    __syncwarp();                                             // the stage that is filled next is no longer read
    if (i + P::STAGES - 1 < n_mine) fetch(i + P::STAGES - 1);
    cp_async_commit();
    cp_async_wait<P::STAGES - 1>();
    __syncwarp();
    const uint32_t sk = ring + (uint32_t)((i % P::STAGES) * P::STAGE), sv = sk + 16 * KD * 2;
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      uint32_t b[4];
      // lanes 0-7: keys 0-7, first half; 8-15: second half; 16-31: keys 8-15 likewise
      ldmatrix_x4(b, sk + page_off<KD>((lane & 7) + (lane >> 4) * 8, k * 2 + ((lane >> 3) & 1)));
      mma_bf16_16816(s[0], q[k], b[0], b[1]);
      mma_bf16_16816(s[1], q[k], b[2], b[3]);
    }
    const int key0 = (p0 + warp + i * kWarps) * 16;
    const bool edge = key0 < first || key0 + 15 > pos;
    float mx[2] = {-CUDART_INF_F, -CUDART_INF_F};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 2 * HR; ++e) {
        const int key = key0 + n * 8 + t4 * 2 + (e & 1);
        float x = s[n][e] * sc - slope[e >> 1] * (float)(pos - key);
        if (edge && (key < first || key > pos)) x = -CUDART_INF_F;
        s[n][e] = x;
        mx[e >> 1] = fmaxf(mx[e >> 1], x);
      }
    bool grow = false;
    float f[2] = {1.f, 1.f};
#pragma unroll
    for (int h = 0; h < HR; ++h) {
      mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
      mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
      if (mx[h] > m[h]) {
        grow = true;
        f[h] = fast_exp2(m[h] - mx[h]);                       // 0 for the first key
        m[h] = mx[h];
      }
    }
    if (__any_sync(0xffffffffu, grow)) {
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 2 * HR; ++e) o[n][e] *= f[e >> 1];
#pragma unroll
      for (int h = 0; h < HR; ++h) l[h] *= f[h];
    }
    uint32_t p[4] = {0u, 0u, 0u, 0u};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int h = 0; h < HR; ++h) {
        const float ref = m[h] == -CUDART_INF_F ? 0.f : m[h];
        const float x = fast_exp2(s[n][2 * h] - ref), y = fast_exp2(s[n][2 * h + 1] - ref);
        l[h] += x + y;
        p[n * 2 + h] = pack_bf162(x, y);
      }
#pragma unroll
    for (int n2 = 0; n2 < NT / 2; ++n2) {
      uint32_t b[4];
      ldmatrix_x4_trans(b, sv + page_off<VD>(lrow, n2 * 2 + lhalf));
      mma_bf16_16816(o[n2 * 2], p, b[0], b[1]);
      mma_bf16_16816(o[n2 * 2 + 1], p, b[2], b[3]);
    }
  }
  cp_async_wait<0>();
  __syncthreads();                                            // the rings become the warps' results

  // ---- merge of the warps ---------------------------------------------------------------------------
  float* mo = reinterpret_cast<float*>(smem);                 // [warp][head][VD]
  float* ml = mo + kWarps * 16 * VD;                          // [warp][head][2]
#pragma unroll
  for (int h = 0; h < HR; ++h) {
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    const int hr = warp * 16 + g + h * 8;
    if (t4 == 0) {
      ml[hr * 2] = m[h];
      ml[hr * 2 + 1] = l[h];
    }
#pragma unroll
    for (int n = 0; n < NT; ++n) *reinterpret_cast<float2*>(mo + hr * VD + n * 8 + t4 * 2) = make_float2(o[n][2 * h], o[n][2 * h + 1]);
  }
  __syncthreads();
  for (int i = tid; i < nh * (VD / 4); i += kThreads) {
    const int h = i / (VD / 4), c = (i - h * (VD / 4)) * 4;
    if (c >= a.vdim) continue;
    float mm = -CUDART_INF_F;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) mm = fmaxf(mm, ml[(w * 16 + h) * 2]);
    float ll = 0.f;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (mm != -CUDART_INF_F) {
#pragma unroll
      for (int w = 0; w < kWarps; ++w) {
        const float f = fast_exp2(ml[(w * 16 + h) * 2] - mm);
        const float4 x = *reinterpret_cast<const float4*>(mo + (w * 16 + h) * VD + c);
        ll += f * ml[(w * 16 + h) * 2 + 1];
        acc.x += f * x.x; acc.y += f * x.y; acc.z += f * x.z; acc.w += f * x.w;
      }
    }
    const int head = h0 + h;
    if (a.splits > 1) {
      const long long at = (row * a.splits + split) * a.heads + head;
      *reinterpret_cast<float4*>(a.part_o + at * a.vdim + c) = acc;
      if (c == 0) {
        a.part_ml[at * 2] = mm;
        a.part_ml[at * 2 + 1] = ll;
      }
      continue;
    }
    const float inv = ll > 0.f ? 1.f / ll : 0.f;
    float gt[4] = {inv, inv, inv, inv};
    if (a.gate != nullptr) {
      const bf16* gp = static_cast<const bf16*>(a.gate) + row * a.gate_stride + (long long)head * a.vdim + c;
#pragma unroll
      for (int j = 0; j < 4; ++j) gt[j] *= sigmoid_f(to_f(gp[j]));
    }
    bf16* out = static_cast<bf16*>(a.out) + row * a.out_stride + (long long)head * a.vdim + c;
    out[0] = hybrid::from_f<bf16>(acc.x * gt[0]);
    out[1] = hybrid::from_f<bf16>(acc.y * gt[1]);
    out[2] = hybrid::from_f<bf16>(acc.z * gt[2]);
    out[3] = hybrid::from_f<bf16>(acc.w * gt[3]);
  }
}

// One thread per output column: the results of a row's key ranges, then the gate.
__global__ void __launch_bounds__(256) kv_merge_kernel(const KvAttentionArgs a) {
  const int cols = a.heads * a.vdim;
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= a.rows * cols) return;
  const long long row = i / cols;
  const int c = (int)(i - row * cols), head = c / a.vdim;
  float m = -CUDART_INF_F, l = 0.f, acc = 0.f;
  for (int s = 0; s < a.splits; ++s) {
    const long long at = (row * a.splits + s) * a.heads + head;
    const float ms = a.part_ml[at * 2];
    if (ms == -CUDART_INF_F) continue;
    const float mn = fmaxf(m, ms), f0 = fast_exp2(m - mn), f1 = fast_exp2(ms - mn);
    l = l * f0 + a.part_ml[at * 2 + 1] * f1;
    acc = acc * f0 + a.part_o[at * a.vdim + c - head * a.vdim] * f1;
    m = mn;
  }
  float y = l > 0.f ? acc / l : 0.f;
  if (a.gate != nullptr) y *= sigmoid_f(to_f(static_cast<const bf16*>(a.gate)[row * a.gate_stride + c]));
  static_cast<bf16*>(a.out)[row * a.out_stride + c] = hybrid::from_f<bf16>(y);
}

template <int KD, int VD, bool HM>
cudaError_t launch_t(const KvAttentionArgs& a, cudaStream_t s) {
  const int rep = a.heads / a.kv_heads, head_blocks = (rep + 15) / 16;
  constexpr int smem = Plan<KD, VD>::BYTES;
  cudaError_t e = cudaFuncSetAttribute(kv_decode_kernel<KD, VD, HM>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  kv_decode_kernel<KD, VD, HM><<<dim3((unsigned)(a.rows * a.splits), (unsigned)(a.kv_heads * head_blocks)), kThreads, smem, s>>>(a, head_blocks);
  e = cudaGetLastError();
  if (e != cudaSuccess || a.splits == 1) return e;
  kv_merge_kernel<<<(unsigned)((a.rows * a.heads * a.vdim + 255) / 256), 256, 0, s>>>(a);
  return cudaGetLastError();
}

template <int KD, int VD>
cudaError_t launch_h(const KvAttentionArgs& a, cudaStream_t s) {
  return a.heads / a.kv_heads <= 8 ? launch_t<KD, VD, true>(a, s) : launch_t<KD, VD, false>(a, s);
}

}  // namespace

bool kv_decode_supported(const KvAttentionArgs& a) {
  const int head_blocks = (a.heads / a.kv_heads + 15) / 16;
  return a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 128 && a.vdim <= 128 && (long long)a.kv_heads * head_blocks < 65536 &&
         (reinterpret_cast<uintptr_t>(a.k_pool) & 15) == 0 && (reinterpret_cast<uintptr_t>(a.v_pool) & 15) == 0 &&
         (reinterpret_cast<uintptr_t>(a.q) & 3) == 0;
}

int kv_decode_splits(long long rows, int kv_heads, int chunk, int max_blocks, int sm_count) {
  long long keys = (long long)max_blocks * 16;
  if (chunk > 0 && chunk < keys) keys = chunk;
  const long long tasks = rows * kv_heads, want = 4ll * sm_count;
  long long n = (want + tasks - 1) / tasks;
  const long long most = keys / 256;                          // a range of at least 256 keys
  if (n > most) n = most;
  return (int)(n < 1 ? 1 : n);
}

cudaError_t launch_kv_decode(const KvAttentionArgs& a, cudaStream_t s) {
  if (a.rows == 0) return cudaSuccess;
  if (a.dim <= 64) return a.vdim <= 64 ? launch_h<64, 64>(a, s) : launch_h<64, 128>(a, s);
  return a.vdim <= 64 ? launch_h<128, 64>(a, s) : launch_h<128, 128>(a, s);
}

}  // namespace mixers
}  // namespace fa
