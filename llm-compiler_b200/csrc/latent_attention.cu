// Latent attention over the cached latents (one row of kv_rank values per token, shared by all heads),
// in the absorbed form: a head's query is carried into the latent space (q W_uk), scored against the
// cached rows themselves, and the weighted sum of the rows is carried out of it (W_uv) behind the
// attention. The softmax denominator may hold a learned term per head (a sink) beside the keys.
//
// This file: the per-head projections in and out of the latent space; attention on warp-level tensor
// cores with the keys split over CTAs (bf16, rank up to 512; B200_LATENT_PATH=mma.sync, the default is
// the tcgen05 kernel of latent_attention_tcgen05.cu), the kernel that combines the splits of either; and
// attention for any rank up to 1024 on the CUDA cores (fp32 models, and shapes the others do not take).
#include <stdlib.h>
#include <string.h>

#include "common.cuh"
#include "hybrid.cuh"
#include "latent_attention.cuh"

namespace b200 {
namespace {

// ---- y[m, h, n] = sum_k x[m, h, k] w[h, n, k] ------------------------------------------------
struct HeadLinearParams {
  const void* x;
  const void* w;
  void* y;
  int m, k, n;
  int64_t x_row_stride, x_head_stride, y_row_stride, y_head_stride;
};

template <typename T>
__global__ void __launch_bounds__(256) head_linear_kernel(const HeadLinearParams p) {
  constexpr int BM = 64, BN = 64, BK = 16;
  __shared__ float As[BK][BM + 4];
  __shared__ float Bs[BK][BN + 4];
  const int m_base = blockIdx.y * BM, n_base = blockIdx.x * BN;
  const T* x = static_cast<const T*>(p.x) + blockIdx.z * p.x_head_stride;
  const T* w = static_cast<const T*>(p.w) + static_cast<int64_t>(blockIdx.z) * p.n * p.k;
  T* y = static_cast<T*>(p.y) + blockIdx.z * p.y_head_stride;
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.k; k0 += BK) {
    for (int id = threadIdx.x; id < BM * BK; id += 256) {
      const int r = id / BK, c = id % BK, kk = k0 + c;
      As[c][r] = m_base + r < p.m && kk < p.k ? Elem<T>::load(x + static_cast<int64_t>(m_base + r) * p.x_row_stride + kk) : 0.0f;
      Bs[c][r] = n_base + r < p.n && kk < p.k ? Elem<T>::load(w + static_cast<int64_t>(n_base + r) * p.k + kk) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < BK; ++kk) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = As[kk][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) b[j] = Bs[kk][tx * 4 + j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m_base + ty * 4 + i, n = n_base + tx * 4 + j;
      if (m < p.m && n < p.n) Elem<T>::store(y + static_cast<int64_t>(m) * p.y_row_stride + n, acc[i][j]);
    }
}

// bf16: 16 or 64 rows x 64 columns of one head per CTA, four warps, a ring of 64-wide k-blocks.
// BM 16: the warps split the columns; BM 64: the rows.
template <int BM>
__global__ void __launch_bounds__(128) head_linear_bf16_kernel(const HeadLinearParams p) {
  constexpr int kStages = 3, BN = 64, BK = 64;
  constexpr int kTilesN = BM == 16 ? 2 : 8;  // n8 tiles of a warp
  constexpr uint32_t kABytes = BM * 128, kStageBytes = kABytes + BN * 128;
  extern __shared__ __align__(128) unsigned char ring[];
  grid_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int m_base = blockIdx.y * BM, n_base = blockIdx.x * BN;
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(p.x) + blockIdx.z * p.x_head_stride;
  const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(p.w) + static_cast<int64_t>(blockIdx.z) * p.n * p.k;
  const uint32_t base = smem_u32(ring);
  const int blocks = (p.k + BK - 1) / BK;
  auto load = [&](int block) {
    const uint32_t stage = base + (block % kStages) * kStageBytes;
    for (int item = threadIdx.x; item < (BM + BN) * 8; item += 128) {
      const int r = item >> 3, chunk = item & 7, kk = block * BK + chunk * 8;
      const bool is_a = r < BM;
      const int row = is_a ? m_base + r : n_base + r - BM;
      const bool inside = row < (is_a ? p.m : p.n) && kk < p.k;
      const __nv_bfloat16* src = is_a ? x + (inside ? static_cast<int64_t>(row) * p.x_row_stride + kk : 0)
                                      : w + (inside ? static_cast<int64_t>(row) * p.k + kk : 0);
      const uint32_t dst = stage + (is_a ? r * 128 : kABytes + (r - BM) * 128);
      cp_async16_zfill(dst + swizzle128(is_a ? r : r - BM, chunk) * 16, src, inside ? 16 : 0);
    }
  };
  grid_dependency_wait_cta();
#pragma unroll
  for (int b = 0; b < kStages - 1; ++b) {
    if (b < blocks) load(b);
    cp_async_commit();
  }
  float acc[kTilesN][4] = {};
  for (int b = 0; b < blocks; ++b) {
    cp_async_wait<kStages - 2>();
    __syncthreads();
    if (b + kStages - 1 < blocks) load(b + kStages - 1);
    cp_async_commit();
    const uint32_t a_tile = base + (b % kStages) * kStageBytes, b_tile = a_tile + kABytes;
    const int a_row = (BM == 16 ? 0 : warp * 16) + (lane & 15);
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t a[4];
      ldmatrix_x4(a, a_tile + a_row * 128 + swizzle128(a_row, ks * 2 + (lane >> 4)) * 16);
#pragma unroll
      for (int pair = 0; pair < kTilesN / 2; ++pair) {
        uint32_t bf[4];  // two n8 tiles x k16
        const int n = (BM == 16 ? warp * 16 : 0) + pair * 16 + ((lane >> 4) << 3) + (lane & 7);
        ldmatrix_x4(bf, b_tile + n * 128 + swizzle128(n, ks * 2 + ((lane >> 3) & 1)) * 16);
        mma_bf16_16816(acc[pair * 2], a, bf[0], bf[1]);
        mma_bf16_16816(acc[pair * 2 + 1], a, bf[2], bf[3]);
      }
    }
  }
  __nv_bfloat16* y = static_cast<__nv_bfloat16*>(p.y) + blockIdx.z * p.y_head_stride;
#pragma unroll
  for (int t = 0; t < kTilesN; ++t) {
    const int n = n_base + (BM == 16 ? warp * 16 : 0) + t * 8 + (lane & 3) * 2;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int m = m_base + (BM == 16 ? 0 : warp * 16) + (lane >> 2) + half * 8;
      if (m >= p.m || n >= p.n) continue;  // n is even and p.n a multiple of 8
      *reinterpret_cast<uint32_t*>(y + static_cast<int64_t>(m) * p.y_row_stride + n) =
          pack_bf16x2(acc[t][half * 2], acc[t][half * 2 + 1]);
    }
  }
}

// ---- attention on the tensor cores ---------------------------------------------------------
// Rows of a sequence are its (token, head) pairs. A CTA takes 16 MT rows and one split of the keys, 32
// keys a step: S = Q C^T (a warp: 8 keys, a quarter of the rank), softmax in fp32 through shared memory,
// O += P C (a warp: a sixteenth of the rank). C, the keys and the values in one, is fetched once for both
// products; the scores of the next step are computed in the same phase as the output of this one. The
// probabilities enter the product as the sum of two bf16 numbers, so that they keep 16 bits of mantissa.
// Splits leave fp32 partial results and (max, sum) pairs; the combining kernel adds the sink to the
// denominator, once.
constexpr int kLatentKeys = 32, kLatentThreads = 512;
constexpr int kScorePitch = kLatentKeys + 4;                  // floats
constexpr int kProbabilityPitch = kLatentKeys * 2 + 16;       // bytes

struct LatentSplitParams {
  const __nv_bfloat16* q;      // [rows, heads, rank]
  const __nv_bfloat16* cache;  // [slots, capacity, rank]
  float* partial;              // [rows * heads, splits, rank]
  float2* partial_stats;       // [rows * heads, splits]: max (log2 domain), sum
  SequenceBatch batch;
  int heads, rank, splits, pitch, stages;  // pitch: bytes of a row in shared memory
  int64_t capacity;
  float scale_log2;
};

template <int MT, int NT>
__global__ void __launch_bounds__(kLatentThreads, 1) latent_attention_split_kernel(const LatentSplitParams p) {
  constexpr int M = 16 * MT;
  extern __shared__ __align__(128) unsigned char smem[];
  __shared__ float row_factor[M];
  __shared__ float row_max[M], row_sum[M];
  grid_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, sequence = blockIdx.z, row0 = blockIdx.y * M;
  grid_dependency_wait_cta();
  const int slot = p.batch.slots[sequence];
  const int first = p.batch.starts[sequence];
  const int rows = (p.batch.starts[sequence + 1] - first) * p.heads;
  if (slot < 0 || row0 >= rows) return;
  const int64_t base = p.batch.bases[sequence];
  const int last_row = min(row0 + M, rows) - 1;
  int64_t keys = base + last_row / p.heads + 1;
  if (keys > p.capacity) keys = p.capacity;
  int64_t begin, end;
  latent_split_range(keys, p.splits, split, kLatentKeys, begin, end);
  const int64_t unit0 = static_cast<int64_t>(first) * p.heads + row0;  // row of q and of the partials
  if (begin >= end) {
    for (int r = threadIdx.x; r <= last_row - row0; r += kLatentThreads)
      p.partial_stats[(unit0 + r) * p.splits + split] = make_float2(-INFINITY, 0.0f);
    return;
  }
  const uint32_t q_tile = smem_u32(smem);
  const uint32_t c_tiles = q_tile + M * p.pitch;
  float* scores = reinterpret_cast<float*>(smem + (M + p.stages * kLatentKeys) * p.pitch);  // [4][M][kScorePitch]
  unsigned char* probabilities = reinterpret_cast<unsigned char*>(scores + 4 * M * kScorePitch);  // [2][M]: high, low
  const int chunks = p.rank / 8;
  for (int item = threadIdx.x; item < M * chunks; item += kLatentThreads) {
    const int r = item / chunks, c = item % chunks;
    const bool inside = row0 + r <= last_row;
    cp_async16_zfill(q_tile + r * p.pitch + c * 16, p.q + (inside ? (unit0 + r) * p.rank + c * 8 : 0), inside ? 16 : 0);
  }
  const __nv_bfloat16* cache = p.cache + static_cast<int64_t>(slot) * p.capacity * p.rank;
  const int steps = static_cast<int>((end - begin + kLatentKeys - 1) / kLatentKeys);
  // a thread copies chunk `copy_chunk` of every `copy_rows`-th key of a step
  const int copy_rows = kLatentThreads / chunks, copy_row = threadIdx.x / chunks, copy_chunk = threadIdx.x - copy_row * chunks;
  auto load = [&](int step, int stage) {
    if (copy_row < copy_rows) {
      const uint32_t tile = c_tiles + stage * kLatentKeys * p.pitch + copy_chunk * 16;
      const int64_t key0 = begin + static_cast<int64_t>(step) * kLatentKeys;
      const __nv_bfloat16* source = cache + key0 * p.rank + copy_chunk * 8;
      const int valid = static_cast<int>(end - key0 < kLatentKeys ? end - key0 : kLatentKeys);
      for (int r = copy_row; r < kLatentKeys; r += copy_rows)
        cp_async16_zfill(tile + r * p.pitch, r < valid ? source + static_cast<int64_t>(r) * p.rank : cache, r < valid ? 16 : 0);
    }
  };
  // tiles 0 .. stages - 2 in flight; one group a tile (the first holds Q as well)
  for (int s = 0; s < p.stages - 1; ++s) {
    if (s < steps) load(s, s);
    cp_async_commit();
  }
  for (int r = threadIdx.x; r < M; r += kLatentThreads) {
    row_max[r] = -INFINITY;
    row_sum[r] = 0.0f;
  }
  const int k_steps = p.rank / 16, quarter = warp >> 2, per_quarter = (k_steps + 3) / 4;
  const int k_begin = quarter * per_quarter, k_end = min(k_begin + per_quarter, k_steps);
  auto compute_scores = [&](uint32_t tile) {
    float s[MT][4] = {};
    const uint32_t b_lane = tile + ((warp & 3) * 8 + (lane & 7)) * p.pitch + ((lane >> 3) & 1) * 16;
    const uint32_t a_lane = q_tile + (lane & 15) * p.pitch + (lane >> 4) * 16;
#pragma unroll 4
    for (int ks = k_begin; ks < k_end; ++ks) {
      uint32_t b[2];
      asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(b[0]), "=r"(b[1]) : "r"(b_lane + ks * 32));
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        uint32_t a[4];
        ldmatrix_x4(a, a_lane + mt * 16 * p.pitch + ks * 32);
        mma_bf16_16816(s[mt], a, b[0], b[1]);
      }
    }
    float* out = scores + quarter * M * kScorePitch + (warp & 3) * 8 + (lane & 3) * 2;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      *reinterpret_cast<float2*>(out + (mt * 16 + (lane >> 2)) * kScorePitch) = make_float2(s[mt][0], s[mt][1]);
      *reinterpret_cast<float2*>(out + (mt * 16 + (lane >> 2) + 8) * kScorePitch) = make_float2(s[mt][2], s[mt][3]);
    }
  };
  float acc[MT][NT][4] = {};
  if (p.stages == 3) cp_async_wait<1>();
  else if (p.stages == 4) cp_async_wait<2>();
  else cp_async_wait<3>();
  __syncthreads();  // tile 0 and Q
  compute_scores(c_tiles);
  int stage = 0;
  for (int step = 0; step < steps; ++step) {
    // tile step + 1 has landed (of the groups behind it, stages - 3 may be in flight)
    if (p.stages == 3) cp_async_wait<0>();
    else if (p.stages == 4) cp_async_wait<1>();
    else cp_async_wait<2>();
    __syncthreads();  // the scores are written; everyone is done with tile step - 1
    const int previous = stage == 0 ? p.stages - 1 : stage - 1;
    if (step + p.stages - 1 < steps) load(step + p.stages - 1, previous);
    cp_async_commit();
    // ---- softmax: 16 lanes a row, 2 keys each ----
    for (int r = threadIdx.x >> 4; r < M; r += kLatentThreads / 16) {
      const int c = (threadIdx.x & 15) * 2;
      float v[2] = {0.0f, 0.0f};
#pragma unroll
      for (int part = 0; part < 4; ++part) {
        const float2 t = *reinterpret_cast<const float2*>(scores + (part * M + r) * kScorePitch + c);
        v[0] += t.x;
        v[1] += t.y;
      }
      const int64_t key0 = begin + static_cast<int64_t>(step) * kLatentKeys + c;
      const int64_t limit = min(base + (row0 + r) / p.heads + 1, end);
      const float before = row_max[r];
      v[0] = key0 < limit ? v[0] * p.scale_log2 : -INFINITY;
      v[1] = key0 + 1 < limit ? v[1] * p.scale_log2 : -INFINITY;
      float top = fmaxf(before, fmaxf(v[0], v[1]));
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
      const float reference = top == -INFINITY ? 0.0f : top;  // (no visible key so far: all weights are 0)
      const float p0 = exp2f(v[0] - reference), p1 = exp2f(v[1] - reference);
      const uint32_t high = pack_bf16x2(p0, p1), low = pack_bf16x2(p0 - bf16_lo(high), p1 - bf16_hi(high));
      float sum = p0 + p1;
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      *reinterpret_cast<uint32_t*>(probabilities + r * kProbabilityPitch + c * 2) = high;
      *reinterpret_cast<uint32_t*>(probabilities + (M + r) * kProbabilityPitch + c * 2) = low;
      if ((threadIdx.x & 15) == 0) {
        const float factor = exp2f(before - reference);  // (0 on the first visible key)
        row_factor[r] = factor;
        row_sum[r] = row_sum[r] * factor + sum;
        row_max[r] = top;
      }
    }
    __syncthreads();
    const uint32_t tile = c_tiles + stage * kLatentKeys * p.pitch;
    stage = stage + 1 == p.stages ? 0 : stage + 1;
    // ---- the next step's scores, and O += P C on this warp's columns ----
    if (step + 1 < steps) compute_scores(c_tiles + stage * kLatentKeys * p.pitch);
    const uint32_t p_tile = smem_u32(probabilities) + (lane & 15) * kProbabilityPitch + (lane >> 4) * 16;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const float f0 = row_factor[mt * 16 + (lane >> 2)], f1 = row_factor[mt * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        acc[mt][t][0] *= f0; acc[mt][t][1] *= f0;
        acc[mt][t][2] *= f1; acc[mt][t][3] *= f1;
      }
    }
#pragma unroll
    for (int ks = 0; ks < kLatentKeys / 16; ++ks) {
      uint32_t hi[MT][4], lo[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        ldmatrix_x4(hi[mt], p_tile + mt * 16 * kProbabilityPitch + ks * 32);
        ldmatrix_x4(lo[mt], p_tile + (M + mt * 16) * kProbabilityPitch + ks * 32);
      }
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        const int n_tile = warp * NT + t;
        if (n_tile < chunks) {
          uint32_t b[2];
          asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];\n"
                       : "=r"(b[0]), "=r"(b[1])
                       : "r"(tile + (ks * 16 + (lane & 15)) * p.pitch + n_tile * 16));
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma_bf16_16816(acc[mt][t], hi[mt], b[0], b[1]);
            mma_bf16_16816(acc[mt][t], lo[mt], b[0], b[1]);
          }
        }
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = mt * 16 + (lane >> 2) + half * 8;
      if (row0 + r > last_row) continue;
      float* out = p.partial + ((unit0 + r) * p.splits + split) * p.rank + (lane & 3) * 2;
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        const int n = (warp * NT + t) * 8;
        if (n < p.rank)
          *reinterpret_cast<float2*>(out + n) = make_float2(acc[mt][t][half * 2], acc[mt][t][half * 2 + 1]);
      }
    }
  for (int r = threadIdx.x; r <= last_row - row0; r += kLatentThreads)  // (written before the last barrier)
    p.partial_stats[(unit0 + r) * p.splits + split] = make_float2(row_max[r], row_sum[r]);
}

// out = sum of the splits' results over (sum of their sums + exp(sink)): one CTA per (row, head)
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* partial, const float2* stats,
                                                             const __nv_bfloat16* sink, __nv_bfloat16* out,
                                                             const SequenceBatch batch, int heads, int rank,
                                                             int splits) {
  grid_launch_dependents();
  grid_dependency_wait_cta();
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * heads + blockIdx.y;
  __nv_bfloat16* dst = out + unit * rank;
  if (batch.slots[batch.token_sequence[blockIdx.x]] < 0) {
    for (int c = threadIdx.x; c < rank; c += blockDim.x) dst[c] = __float2bfloat16_rn(0.0f);
    return;
  }
  const float own = sink != nullptr ? __bfloat162float(sink[blockIdx.y]) * 1.4426950408889634f : -INFINITY;
  float top = own;
  for (int s = 0; s < splits; ++s) top = fmaxf(top, stats[unit * splits + s].x);
  float total = exp2f(own - top);
  for (int s = 0; s < splits; ++s) {
    const float2 st = stats[unit * splits + s];
    total += st.y * exp2f(st.x - top);
  }
  const float inverse = 1.0f / total;
  for (int c = threadIdx.x * 2; c < rank; c += blockDim.x * 2) {
    float a = 0.0f, b = 0.0f;
    for (int s = 0; s < splits; ++s) {
      const float2 st = stats[unit * splits + s];
      if (st.y == 0.0f) continue;  // a split without keys left no result
      const float f = exp2f(st.x - top);
      const float2 v = *reinterpret_cast<const float2*>(partial + (unit * splits + s) * rank + c);
      a = fmaf(v.x, f, a);
      b = fmaf(v.y, f, b);
    }
    *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(a * inverse, b * inverse);
  }
}

struct LatentPlan {
  int mt, nt, row_blocks, splits, pitch, stages, smem;
};

// Row tile, ring depth and split count: as many CTAs as fill the GPU's slots in whole waves.
LatentPlan plan_latent(int64_t sequences, int64_t longest, int64_t heads, int64_t rank, int64_t context) {
  LatentPlan plan{};
  if (rank % 16 != 0 || rank > 512) return plan;
  const int64_t rows = longest * heads;
  plan.mt = rows <= 16 ? 1 : rows <= 32 ? 2 : 4;
  plan.nt = rank <= 128 ? 1 : rank <= 256 ? 2 : 4;
  const int m = 16 * plan.mt;
  plan.pitch = static_cast<int>(rank * 2 + 16);
  const int fixed = m * plan.pitch + 4 * m * kScorePitch * 4 + 2 * m * kProbabilityPitch;
  for (plan.stages = 5; plan.stages > 3; --plan.stages)
    if (fixed + plan.stages * kLatentKeys * plan.pitch <= 224 * 1024) break;
  plan.smem = fixed + plan.stages * kLatentKeys * plan.pitch;
  if (plan.smem > 224 * 1024) return LatentPlan{};
  plan.row_blocks = static_cast<int>(ceil_div(rows, m));
  const int64_t slots = kNumSMs, units = sequences * plan.row_blocks;
  const int64_t most = ceil_div(context, 128);
  double best = -1.0;
  plan.splits = 1;
  for (int64_t s = 1; s <= 64 && s <= most; ++s) {
    const int64_t ctas = units * s;
    const double fill = static_cast<double>(ctas) / (ceil_div(ctas, slots) * slots) - 0.01 * s;
    if (fill > best) {
      best = fill;
      plan.splits = static_cast<int>(s);
    }
  }
  return plan;
}

template <int MT, int NT>
int launch_split(const LatentSplitParams& p, const LatentPlan& plan, int64_t sequences, cudaStream_t stream) {
  auto kernel = latent_attention_split_kernel<MT, NT>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, plan.smem) != cudaSuccess)
    return B200_ERR_LAUNCH;
  const dim3 grid(static_cast<unsigned>(plan.splits), static_cast<unsigned>(plan.row_blocks),
                  static_cast<unsigned>(sequences));
  return launch_chained(kernel, grid, dim3(kLatentThreads), plan.smem, stream, p) == cudaSuccess ? B200_OK
                                                                                                : B200_ERR_LAUNCH;
}
template <int MT>
int launch_split_nt(const LatentSplitParams& p, const LatentPlan& plan, int64_t sequences, cudaStream_t stream) {
  switch (plan.nt) {
    case 1: return launch_split<MT, 1>(p, plan, sequences, stream);
    case 2: return launch_split<MT, 2>(p, plan, sequences, stream);
    default: return launch_split<MT, 4>(p, plan, sequences, stream);
  }
}

// ---- attention on the CUDA cores -----------------------------------------------------------
struct LatentAttentionParams {
  const void* q;      // T [rows, heads, rank_row]
  const void* cache;  // T [slots, capacity, rank_row]
  const void* sink;   // T [heads] or NULL
  void* out;          // T [rows, heads, rank_row]
  SequenceBatch batch;
  int heads, rank_row;
  int64_t capacity;
  float scale;
};

// One CTA per (head, row); four warps take every fourth group of four keys, a lane every 32nd dimension.
template <typename T, int R>
__global__ void __launch_bounds__(128) latent_attention_generic_kernel(const LatentAttentionParams p) {
  constexpr int kWarps = 4, kKeys = 4;
  __shared__ float merge_max[kWarps], merge_sum[kWarps];
  extern __shared__ float merge_acc[];  // [kWarps][rank_row]
  const int head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t row = blockIdx.x;
  const int sequence = p.batch.token_sequence[row];
  const int slot = p.batch.slots[sequence];
  T* out = static_cast<T*>(p.out) + (row * p.heads + head) * p.rank_row;
  if (slot < 0) {
    for (int c = threadIdx.x; c < p.rank_row; c += blockDim.x) Elem<T>::store(out + c, 0.0f);
    return;
  }
  int64_t keys = p.batch.position(sequence, row) + 1;
  if (keys > p.capacity) keys = p.capacity;
  const T* q = static_cast<const T*>(p.q) + (row * p.heads + head) * p.rank_row;
  const T* cache = static_cast<const T*>(p.cache) + static_cast<int64_t>(slot) * p.capacity * p.rank_row;
  float qr[R], acc[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = lane + 32 * i;
    qr[i] = c < p.rank_row ? Elem<T>::load(q + c) : 0.0f;
    acc[i] = 0.0f;
  }
  float top = -INFINITY, sum = 0.0f;
  for (int64_t key0 = warp * kKeys; key0 < keys; key0 += kWarps * kKeys) {
    float value[kKeys][R], score[kKeys];
#pragma unroll
    for (int j = 0; j < kKeys; ++j) {
      score[j] = 0.0f;
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int c = lane + 32 * i;
        value[j][i] = key0 + j < keys && c < p.rank_row ? Elem<T>::load(cache + (key0 + j) * p.rank_row + c) : 0.0f;
        score[j] = fmaf(qr[i], value[j][i], score[j]);
      }
    }
    float group_top = top;
#pragma unroll
    for (int j = 0; j < kKeys; ++j) {
      score[j] = key0 + j < keys ? warp_sum(score[j]) * p.scale : -INFINITY;
      group_top = fmaxf(group_top, score[j]);
    }
    const float factor = expf(top - group_top);
    top = group_top;
    sum *= factor;
#pragma unroll
    for (int i = 0; i < R; ++i) acc[i] *= factor;
#pragma unroll
    for (int j = 0; j < kKeys; ++j) {
      const float weight = expf(score[j] - top);
      sum += weight;
#pragma unroll
      for (int i = 0; i < R; ++i) acc[i] = fmaf(weight, value[j][i], acc[i]);
    }
  }
  if (lane == 0) {
    merge_max[warp] = top;
    merge_sum[warp] = sum;
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = lane + 32 * i;
    if (c < p.rank_row) merge_acc[warp * p.rank_row + c] = acc[i];
  }
  __syncthreads();
  const float sink = p.sink != nullptr ? Elem<T>::load(static_cast<const T*>(p.sink) + head) : -INFINITY;
  float all = sink;
  for (int w = 0; w < kWarps; ++w) all = fmaxf(all, merge_max[w]);
  float total = expf(sink - all);
  float factors[kWarps];
#pragma unroll
  for (int w = 0; w < kWarps; ++w) {
    factors[w] = expf(merge_max[w] - all);
    total += merge_sum[w] * factors[w];
  }
  for (int c = threadIdx.x; c < p.rank_row; c += blockDim.x) {
    float v = 0.0f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) v += merge_acc[w * p.rank_row + c] * factors[w];
    Elem<T>::store(out + c, v / total);
  }
}

template <typename T>
int launch_generic(const LatentAttentionParams& p, int64_t rows, cudaStream_t stream) {
  const dim3 grid(static_cast<unsigned>(rows), static_cast<unsigned>(p.heads));
  const size_t smem = 4 * p.rank_row * sizeof(float);
  if (p.rank_row <= 64) latent_attention_generic_kernel<T, 2><<<grid, 128, smem, stream>>>(p);
  else if (p.rank_row <= 128) latent_attention_generic_kernel<T, 4><<<grid, 128, smem, stream>>>(p);
  else if (p.rank_row <= 256) latent_attention_generic_kernel<T, 8><<<grid, 128, smem, stream>>>(p);
  else if (p.rank_row <= 512) latent_attention_generic_kernel<T, 16><<<grid, 128, smem, stream>>>(p);
  else if (p.rank_row <= 1024) latent_attention_generic_kernel<T, 32><<<grid, 128, smem, stream>>>(p);
  else return B200_ERR_TOO_LARGE;
  return launch_status();
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int b200_head_linear(const void* x, const void* w, void* y, int64_t m, int64_t heads, int64_t k,
                                int64_t n, int64_t x_row_stride, int64_t x_head_stride, int64_t y_row_stride,
                                int64_t y_head_stride, int dtype, void* stream) {
  if (!x || !w || !y || m < 0 || heads <= 0 || k <= 0 || n <= 0) return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (m == 0) return B200_OK;
  const dim3 grid(static_cast<unsigned>(ceil_div(n, 64)), static_cast<unsigned>(ceil_div(m, 64)),
                  static_cast<unsigned>(heads));
  if (grid.y > 65535 || heads > 65535) return B200_ERR_TOO_LARGE;
  HeadLinearParams p{x, w, y, static_cast<int>(m), static_cast<int>(k), static_cast<int>(n), x_row_stride,
                     x_head_stride, y_row_stride, y_head_stride};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  // 16-byte rows and chunks: the tensor-core kernel
  if (dtype == B200_BF16 && k % 8 == 0 && n % 8 == 0 && x_row_stride % 8 == 0 && x_head_stride % 8 == 0 &&
      y_row_stride % 2 == 0 && y_head_stride % 2 == 0 && aligned16(x) && aligned16(w) && aligned16(y)) {
    const int bm = m <= 16 ? 16 : 64;
    const dim3 tiles(static_cast<unsigned>(ceil_div(n, 64)), static_cast<unsigned>(ceil_div(m, bm)),
                     static_cast<unsigned>(heads));
    const int smem = 3 * (bm + 64) * 128;
    auto kernel = bm == 16 ? head_linear_bf16_kernel<16> : head_linear_bf16_kernel<64>;
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return B200_ERR_LAUNCH;
    return launch_chained(kernel, tiles, dim3(128), smem, s, p) == cudaSuccess ? launch_status() : B200_ERR_LAUNCH;
  }
  if (dtype == B200_F32) head_linear_kernel<float><<<grid, 256, 0, s>>>(p);
  else head_linear_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(p);
  return launch_status();
}

// Which split-KV kernel serves a bf16 call, and with how many splits; splits 0: neither does.
struct LatentChoice {
  LatentTcPlan tcgen05;
  LatentPlan warp_level;
  int splits;
};
static LatentChoice choose_latent(int64_t sequences, int64_t longest, int64_t heads, int64_t rank, int64_t context) {
  LatentChoice choice{};
  const char* path = getenv("B200_LATENT_PATH");
  if (path == nullptr || strcmp(path, "mma.sync") != 0)
    choice.tcgen05 = plan_latent_tcgen05(sequences, longest, heads, rank, context);
  choice.splits = choice.tcgen05.splits;
  if (choice.tcgen05.n == 0) {
    choice.warp_level = plan_latent(sequences, longest, heads, rank, context);
    choice.splits = choice.warp_level.mt != 0 ? choice.warp_level.splits : 0;
  }
  return choice;
}

extern "C" int64_t b200_latent_attention_workspace_bytes(int64_t rows, int64_t sequences, int64_t longest,
                                                         int64_t heads, int64_t rank_row, int64_t context,
                                                         int dtype) {
  if (dtype != B200_BF16 || rows <= 0 || sequences <= 0 || longest <= 0 || heads <= 0 || rank_row <= 0 || context <= 0)
    return 0;
  return rows * heads * choose_latent(sequences, longest, heads, rank_row, context).splits * (rank_row + 2) * 4;
}

extern "C" int b200_latent_attention(const void* q, const void* cache, const void* sink, void* out,
                                     const int32_t* token_sequence, const int32_t* starts, const int32_t* slots,
                                     const int32_t* bases, int64_t rows, int64_t sequences, int64_t longest,
                                     int64_t heads, int64_t rank_row, int64_t slot_count, int64_t capacity,
                                     int64_t context, double scale, int dtype, void* workspace,
                                     int64_t workspace_bytes, int32_t* status, void* stream) {
  if (!q || !cache || !out || !token_sequence || !starts || !slots || !bases || rows < 0 || sequences <= 0 ||
      longest <= 0 || heads <= 0 || rank_row <= 0 || slot_count <= 0 || capacity <= 0 || context <= 0)
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (rows * heads > INT32_MAX || heads > 65535 || sequences > 65535) return B200_ERR_TOO_LARGE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const SequenceBatch batch{token_sequence, starts, slots, bases};
  const LatentChoice choice = dtype == B200_BF16 ? choose_latent(sequences, longest, heads, rank_row, context) : LatentChoice{};
  if (choice.splits > 0) {
    const int64_t need = rows * heads * choice.splits * (rank_row + 2) * 4;
    if (!workspace || workspace_bytes < need) return B200_ERR_WORKSPACE;
    if (!aligned16(q) || !aligned16(cache) || !aligned16(workspace)) return B200_ERR_ALIGNMENT;
    float* partial = static_cast<float*>(workspace);
    float2* stats = reinterpret_cast<float2*>(partial + rows * heads * choice.splits * rank_row);
    int code;
    if (choice.tcgen05.n != 0) {
      if (choice.tcgen05.row_blocks > 65535) return B200_ERR_TOO_LARGE;
      code = latent_attention_tcgen05(choice.tcgen05, q, cache, partial, stats, batch, rows, sequences, heads, rank_row,
                                      slot_count, capacity, scale, status, s);
    } else {
      const LatentPlan& plan = choice.warp_level;
      if (plan.row_blocks > 65535) return B200_ERR_TOO_LARGE;
      LatentSplitParams p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(cache), partial, stats,
                          batch, static_cast<int>(heads), static_cast<int>(rank_row), plan.splits, plan.pitch, plan.stages,
                          capacity, static_cast<float>(scale * 1.4426950408889634)};
      code = plan.mt == 1 ? launch_split_nt<1>(p, plan, sequences, s)
             : plan.mt == 2 ? launch_split_nt<2>(p, plan, sequences, s)
                            : launch_split_nt<4>(p, plan, sequences, s);
    }
    if (code != B200_OK) return code;
    const dim3 grid(static_cast<unsigned>(rows), static_cast<unsigned>(heads));
    return launch_chained(latent_combine_kernel, grid, dim3(128), 0, s, static_cast<const float*>(partial),
                          static_cast<const float2*>(stats), static_cast<const __nv_bfloat16*>(sink),
                          static_cast<__nv_bfloat16*>(out), batch, static_cast<int>(heads),
                          static_cast<int>(rank_row), choice.splits) == cudaSuccess
               ? launch_status() : B200_ERR_LAUNCH;
  }
  LatentAttentionParams p{q, cache, sink, out, batch, static_cast<int>(heads),
                          static_cast<int>(rank_row), capacity, static_cast<float>(scale)};
  return dtype == B200_F32 ? launch_generic<float>(p, rows, s) : launch_generic<__nv_bfloat16>(p, rows, s);
}
