// Latent attention over cached latents on the 5th-generation tensor cores, transposed: the 128 keys of a
// tile are the M rows of the score product and the rank is the M extent of the output product, so that
// both run at full width however few (token, head) rows a decode step has; those rows are N (32 or 64).
//
//   S^T [128 keys x N]       = C Q^T        C tile K-major (as TMA lays it down), Q K-major
//   O^T [128 rank x N] each  = C^T P^T      the same C tile read MN-major, P [N x 128 keys] K-major
//
// so one read of HBM serves as key and as value. The tile is cut into pairs of 64-column panels (32 KB) that
// stream through a ring. Where the ring holds two tiles, a tile's pairs stay until its output product has
// read them. Where it does not (rank above 256), every pair is fetched twice, once per product (the second
// time from L2, a few microseconds later), so that the stream never waits for a softmax: the scores of tile
// j + 1 are computed before the output of tile j. One thread issues the TMA boxes, one the MMAs; four warps
// hold a key per thread, take the column maxima with warp reductions, and write the probabilities as two
// bf16 numbers whose sum keeps 16 bits of mantissa: both are rows of one operand (2 N columns of O^T, added at
// the end), because a product of this shape costs what reading its M operand costs. The reference maximum is lazy: O^T is rescaled in tensor memory only when a row's
// maximum rises by more than 8 in the log2 domain. Every wait is bounded.
#include "common.cuh"
#include "hybrid.cuh"
#include "latent_attention.cuh"
#include "tcgen05.cuh"
#include "tensor_map.cuh"

namespace b200 {
namespace {

constexpr int kTileKeys = 128, kPanelBytes = kTileKeys * 128, kPairBytes = 2 * kPanelBytes;
constexpr int kMaxRing = 6;
constexpr int kSoftmaxWarps = 4, kTmaWarp = 4, kMmaWarp = 5, kThreads = 192;
constexpr float kRaise = 8.0f;  // log2 domain

struct LatentTcParams {
  float* partial;         // [rows * heads, splits, rank]
  float2* partial_stats;  // [rows * heads, splits]: reference (log2 domain), sum
  SequenceBatch batch;
  int32_t* status;
  int heads, rank, splits, pairs, ring, refetch;
  int64_t capacity;
  float scale_log2;
  uint32_t wait_limit;
  int drop_loads;
};

__device__ __forceinline__ float exp2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Maximum over the warp: floats as integers of the same order
__device__ __forceinline__ float warp_max_redux(float v) {
  int i = __float_as_int(v);
  i ^= (i >> 31) & 0x7fffffff;
  i = __reduce_max_sync(0xffffffffu, i);
  i ^= (i >> 31) & 0x7fffffff;
  return __int_as_float(i);
}

template <int N>
__global__ void __launch_bounds__(kThreads, 1)
latent_attention_tcgen05_kernel(const LatentTcParams p, const __grid_constant__ CUtensorMap q_map,
                                const __grid_constant__ CUtensorMap c_map) {
  constexpr int kGroups = N / 32;                        // 32-column groups of a row of S^T
  constexpr uint32_t kQPanel = N * 128, kPPanel = 2 * N * 128, kPLow = N * 128;
  extern __shared__ __align__(1024) unsigned char smem[];
  __shared__ __align__(8) uint64_t q_full, s_full[2], p_full, o_done, pair_full[kMaxRing], pair_empty[kMaxRing];
  __shared__ float warp_tops[2][kSoftmaxWarps][N];
  __shared__ int limits[N];
  __shared__ uint32_t tmem_slot;
  __shared__ int failed;
  grid_launch_dependents();
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  const int split = blockIdx.x, sequence = blockIdx.z, row0 = blockIdx.y * N;
  const uint32_t columns = (p.pairs + 2) * 2 * N <= 256 ? 256u : 512u;
  if (threadIdx.x == 0) {
    failed = 0;
    mbarrier_init(smem_u32(&q_full), 1);
    mbarrier_init(smem_u32(&s_full[0]), 1);
    mbarrier_init(smem_u32(&s_full[1]), 1);
    mbarrier_init(smem_u32(&p_full), kSoftmaxWarps);
    mbarrier_init(smem_u32(&o_done), 1);
    for (int i = 0; i < kMaxRing; ++i) {
      mbarrier_init(smem_u32(&pair_full[i]), 1);
      mbarrier_init(smem_u32(&pair_empty[i]), 1);
    }
    fence_mbarrier_init();
  }
  if (warp == kTmaWarp && lane == 0) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&q_map)) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&c_map)) : "memory");
  }
  if (warp == kMmaWarp) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;"
                 ::"r"(smem_u32(&tmem_slot)), "r"(columns) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  grid_dependency_wait_cta();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = tmem_slot;

  const int slot = p.batch.slots[sequence];
  const int first = p.batch.starts[sequence];
  const int rows = (p.batch.starts[sequence + 1] - first) * p.heads;
  const int64_t base = p.batch.bases[sequence];
  const int last_row = min(row0 + N, rows) - 1;
  int64_t keys = base + last_row / p.heads + 1;
  if (keys > p.capacity) keys = p.capacity;
  int64_t begin = 0, end = 0;
  if (slot >= 0 && row0 < rows) latent_split_range(keys, p.splits, split, kTileKeys, begin, end);
  const bool active = begin < end;
  const int64_t unit0 = static_cast<int64_t>(first) * p.heads + row0;  // row of q and of the partials
  const int span = static_cast<int>(end - begin);                      // keys of this split
  const int tiles = (span + kTileKeys - 1) / kTileKeys;
  const uint32_t ring_smem = smem_u32(smem);
  const uint32_t q_smem = ring_smem + p.ring * kPairBytes;             // [2 pairs] panels of N rows
  const uint32_t p_smem = q_smem + 2 * p.pairs * kQPanel;              // [2 panels of 64 keys][N high, N low rows]
  const uint32_t o_column = tmem + 4 * N;  // behind two buffers of two partial S^T
  if (active && threadIdx.x < N)  // first key, counted from begin, that a row does not see
    limits[threadIdx.x] = row0 + static_cast<int>(threadIdx.x) <= last_row
                              ? static_cast<int>(min(base + (row0 + static_cast<int>(threadIdx.x)) / p.heads + 1, end) - begin)
                              : 0;
  __syncthreads();

  if (!active) {
    if (slot >= 0 && row0 < rows)
      for (int r = threadIdx.x; r <= last_row - row0; r += kThreads)
        p.partial_stats[(unit0 + r) * p.splits + split] = make_float2(-INFINITY, 0.0f);
  } else if (warp == kTmaWarp && lane == 0 && !p.drop_loads) {
    // ---- TMA producer ----
    mbarrier_arrive_expect_tx(smem_u32(&q_full), 2 * p.pairs * kQPanel);
    for (int panel = 0; panel < 2 * p.pairs; ++panel)
      tma_load_2d(q_smem + panel * kQPanel, &q_map, smem_u32(&q_full), panel * 64, static_cast<int>(unit0));
    bool ok = true;
    int index = 0;  // pairs fetched so far
    auto push = [&](int j) {
      for (int m = 0; ok && m < p.pairs; ++m) {
        const int place = index % p.ring, use = index / p.ring;
        ok = use == 0 || mbarrier_wait_bounded(smem_u32(&pair_empty[place]), (use - 1) & 1, p.wait_limit);
        if (!ok) return;
        mbarrier_arrive_expect_tx(smem_u32(&pair_full[place]), kPairBytes);
        for (int half = 0; half < 2; ++half)
          tma_load_3d(ring_smem + place * kPairBytes + half * kPanelBytes, &c_map, smem_u32(&pair_full[place]),
                      m * 128 + half * 64, static_cast<int>(begin) + j * kTileKeys, slot);
        ++index;
      }
    };
    push(0);
    for (int j = 0; ok && j < tiles; ++j) {
      if (j + 1 < tiles) push(j + 1);
      if (p.refetch) push(j);
    }
    if (!ok) failed = 1;
    // nothing of this CTA's is in flight when it ends
    mbarrier_wait_bounded(smem_u32(&q_full), 0, p.wait_limit);
    for (int i = max(0, index - p.ring); i < index; ++i)
      mbarrier_wait_bounded(smem_u32(&pair_full[i % p.ring]), (i / p.ring) & 1, p.wait_limit);
  } else if (warp == kMmaWarp) {
    // ---- MMA issuer: the whole warp walks the loops (the descriptors stay in uniform registers), one lane issues ----
    const uint32_t leader = lane == 0 ? 1u : 0u;
    constexpr uint32_t idesc_s = instruction_descriptor(128, N);
    constexpr uint32_t idesc_o = instruction_descriptor(128, 2 * N, false, true);
    const uint64_t q_desc = smem_descriptor(q_smem), p_desc = smem_descriptor(p_smem);
    bool ok = __all_sync(0xffffffffu, mbarrier_wait_bounded(smem_u32(&q_full), 0, p.wait_limit));
    int index = 0;  // pairs taken so far (refetch)
    auto next_pair = [&](int j, int m) { return p.refetch ? index++ : j * p.pairs + m; };
    auto landed = [&](int pair) {
      ok = __all_sync(0xffffffffu, mbarrier_wait_bounded(smem_u32(&pair_full[pair % p.ring]), (pair / p.ring) & 1, p.wait_limit));
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      return ok;
    };
    auto issue_scores = [&](int j) {
      for (int m = 0; m < p.pairs; ++m) {
        const int pair = next_pair(j, m);
        if (!landed(pair)) return;
        const uint64_t c_desc = smem_descriptor(ring_smem + pair % p.ring * kPairBytes);
#pragma unroll
        for (int ks = 0; ks < 8; ++ks)
          umma_bf16_if(leader, tmem + ((j & 1) * 2 + (ks & 1)) * N, descriptor_advance(c_desc, (ks / 4) * kPanelBytes + (ks % 4) * 32),
                    descriptor_advance(q_desc, (2 * m + ks / 4) * kQPanel + (ks % 4) * 32), idesc_s,
                    m > 0 || ks > 1 ? 1u : 0u);
        if (p.refetch) umma_commit_if(leader, smem_u32(&pair_empty[pair % p.ring]));
      }
      umma_commit_if(leader, smem_u32(&s_full[j & 1]));
    };
    if (ok) issue_scores(0);
    for (int j = 0; ok && j < tiles; ++j) {
      if (j + 1 < tiles) issue_scores(j + 1);  // (its buffer's scores, of tile j - 1, were read before p_full of j - 1)
      ok = ok && __all_sync(0xffffffffu, mbarrier_wait_bounded(smem_u32(&p_full), j & 1, p.wait_limit));
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      // Products with one accumulator follow one another at the latency of a product: two blocks of O^T
      // take turns.
      for (int m = 0; ok && m < p.pairs; m += 2) {
        const bool two = m + 1 < p.pairs;
        const int pair0 = next_pair(j, m), pair1 = two ? next_pair(j, m + 1) : pair0;
        if (p.refetch && (!landed(pair0) || (two && !landed(pair1)))) break;
        const uint64_t c0 = smem_descriptor_mn_major(ring_smem + pair0 % p.ring * kPairBytes, kPanelBytes);
        const uint64_t c1 = smem_descriptor_mn_major(ring_smem + pair1 % p.ring * kPairBytes, kPanelBytes);
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {  // 16 keys a step
          const uint32_t at = (ks / 4) * kPPanel + (ks % 4) * 32, accumulate = j > 0 || ks > 0 ? 1u : 0u;
          umma_bf16_if(leader, o_column + m * 2 * N, descriptor_advance(c0, ks * 2048), descriptor_advance(p_desc, at), idesc_o, accumulate);
          if (two)
            umma_bf16_if(leader, o_column + (m + 1) * 2 * N, descriptor_advance(c1, ks * 2048), descriptor_advance(p_desc, at), idesc_o,
                      accumulate);
        }
        umma_commit_if(leader, smem_u32(&pair_empty[pair0 % p.ring]));
        if (two) umma_commit_if(leader, smem_u32(&pair_empty[pair1 % p.ring]));
      }
      if (ok) umma_commit_if(leader, smem_u32(&o_done));
    }
    if (!ok) failed = 1;
  } else if (warp < kSoftmaxWarps) {
    // ---- softmax: one key a thread ----
    const int row = warp * 32 + lane;                               // key of the tile, lane of tensor memory
    const uint32_t lane_base = static_cast<uint32_t>(warp * 32) << 16;
    float reference[kGroups];                                       // of row 32 g + lane
    float sums[N];                                                  // over this thread's keys
#pragma unroll
    for (int g = 0; g < kGroups; ++g) reference[g] = -INFINITY;
#pragma unroll
    for (int n = 0; n < N; ++n) sums[n] = 0.0f;
    int seen_by_all = limits[0];  // keys below it are seen by every row
    for (int n = 1; n <= last_row - row0; ++n) seen_by_all = min(seen_by_all, limits[n]);
    const uint32_t p_row = p_smem + (row >> 6) * kPPanel + (row & 7) * 2;
    const uint32_t chunk = (row & 63) >> 3;
    bool ok = true;
    for (int j = 0; j < tiles; ++j) {
      ok = ok && __all_sync(0xffffffffu, mbarrier_wait_ready_first(smem_u32(&s_full[j & 1]), (j >> 1) & 1, p.wait_limit));
      float s[N];
      const int key = j * kTileKeys + row;
      if (ok) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
        for (int g = 0; g < kGroups; ++g) {
          float t[32], u[32];  // the sums over even and odd k-steps
          tmem_load_32x32(tmem + (j & 1) * 2 * N + lane_base + g * 32, t);
          tmem_load_32x32(tmem + (j & 1) * 2 * N + N + lane_base + g * 32, u);
#pragma unroll
          for (int i = 0; i < 32; ++i) s[g * 32 + i] = (t[i] + u[i]) * p.scale_log2;
        }
        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
        if ((j + 1) * kTileKeys > seen_by_all) {
#pragma unroll
          for (int n = 0; n < N; ++n)
            if (key >= limits[n]) s[n] = -INFINITY;
        }
#pragma unroll
        for (int g = 0; g < kGroups; ++g) {
          float top = 0.0f;
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float t = warp_max_redux(s[g * 32 + i]);
            if (lane == i) top = t;
          }
          warp_tops[j & 1][warp][g * 32 + lane] = top;
        }
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      if (!ok) continue;
      // every warp moves its copy of the references alike
      float factor[kGroups];
      bool raise = false;
#pragma unroll
      for (int g = 0; g < kGroups; ++g) {
        float top = warp_tops[j & 1][0][g * 32 + lane];
#pragma unroll
        for (int w = 1; w < kSoftmaxWarps; ++w) top = fmaxf(top, warp_tops[j & 1][w][g * 32 + lane]);
        const bool move = top > reference[g] + kRaise || (reference[g] == -INFINITY && top > -INFINITY);
        factor[g] = move ? exp2_fast(reference[g] - top) : 1.0f;  // (0 where nothing had been seen)
        if (move) reference[g] = top;
        raise = raise || move;
      }
      raise = __any_sync(0xffffffffu, raise);
      // the probabilities' planes and O^T are in use until the previous tile's products have retired
      if (j > 0) ok = __all_sync(0xffffffffu, mbarrier_wait_ready_first(smem_u32(&o_done), (j - 1) & 1, p.wait_limit));
      if (!ok) continue;
      if (raise && j > 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
        for (int g = 0; g < kGroups; ++g) {
          float f[32];
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            f[i] = __shfl_sync(0xffffffffu, factor[g], i);
            sums[g * 32 + i] *= f[i];
          }
          for (int m = 0; m < 2 * p.pairs; ++m) {  // high and low parts
            float t[32];
            tmem_load_32x32(o_column + m * N + lane_base + g * 32, t);
#pragma unroll
            for (int i = 0; i < 32; ++i) t[i] *= f[i];
            tmem_store_32x32(o_column + m * N + lane_base + g * 32, t);
          }
        }
        tmem_store_wait();
      }
#pragma unroll
      for (int n = 0; n < N; ++n) {
        const float r = __shfl_sync(0xffffffffu, reference[n / 32], n % 32);
        const float value = exp2_fast(s[n] - (r == -INFINITY ? 0.0f : r));
        sums[n] += value;
        const uint16_t high = f32_to_bf16_bits(value), low = f32_to_bf16_bits(value - bf16_to_f32(high));
        const uint32_t at = p_row + n * 128 + ((chunk ^ (n & 7)) << 4);
        asm volatile("st.shared.u16 [%0], %1;" ::"r"(at), "h"(high) : "memory");
        asm volatile("st.shared.u16 [%0], %1;" ::"r"(at + kPLow), "h"(low) : "memory");
      }
      if ((j + 1) * kTileKeys > span) {  // rows behind the split's end carry weight 0: make them 0 as values, too
        for (int m = 0; m < p.pairs; ++m) {
          const int pair = p.refetch ? (2 * tiles - 1) * p.pairs + m : j * p.pairs + m;
          if (p.refetch)
            ok = ok && __all_sync(0xffffffffu, mbarrier_wait_ready_first(smem_u32(&pair_full[pair % p.ring]),
                                                                         (pair / p.ring) & 1, p.wait_limit));
          if (!ok || key < span) continue;
          const uint32_t at = ring_smem + pair % p.ring * kPairBytes + row * 128;
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};" ::"r"(at + i * 16), "r"(0u) : "memory");
            asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};" ::"r"(at + kPanelBytes + i * 16), "r"(0u) : "memory");
          }
        }
        if (!ok) continue;
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&p_full)) : "memory");
    }
    ok = ok && __all_sync(0xffffffffu, mbarrier_wait_ready_first(smem_u32(&o_done), (tiles - 1) & 1, p.wait_limit));
    if (!ok) {
      failed = 1;
    } else {
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      for (int m = 0; m < p.pairs; ++m)
#pragma unroll
        for (int g = 0; g < kGroups; ++g) {
          float t[32], low[32];
          tmem_load_32x32(o_column + m * 2 * N + lane_base + g * 32, t);
          tmem_load_32x32(o_column + m * 2 * N + N + lane_base + g * 32, low);
          if (m * 128 + row < p.rank) {
            float* out = p.partial + ((unit0 + g * 32) * p.splits + split) * p.rank + m * 128 + row;
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (row0 + g * 32 + i <= last_row) out[static_cast<int64_t>(i) * p.splits * p.rank] = t[i] + low[i];
          }
        }
    }
    // sums over the keys: over the warp, then over the four warps
#pragma unroll
    for (int g = 0; g < kGroups; ++g) {
      float total = 0.0f;
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        const float t = warp_sum(sums[g * 32 + i]);
        if (lane == i) total = t;
      }
      warp_tops[tiles & 1][warp][g * 32 + lane] = total;
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    if (warp == 0 && ok) {
#pragma unroll
      for (int g = 0; g < kGroups; ++g) {
        float total = 0.0f;
#pragma unroll
        for (int w = 0; w < kSoftmaxWarps; ++w) total += warp_tops[tiles & 1][w][g * 32 + lane];
        if (row0 + g * 32 + lane <= last_row)
          p.partial_stats[(unit0 + g * 32 + lane) * p.splits + split] = make_float2(reference[g], total);
      }
    }
  }
  __syncwarp();
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (failed && threadIdx.x == 0 && p.status != nullptr) atomicOr(p.status, B200_STATUS_WAIT_TIMEOUT);
  if (warp == kMmaWarp)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(columns) : "memory");
}

}  // namespace

LatentTcPlan plan_latent_tcgen05(int64_t sequences, int64_t longest, int64_t heads, int64_t rank, int64_t context) {
  LatentTcPlan plan{};
  if (rank % 16 != 0 || rank > 512) return plan;
  const int64_t rows = longest * heads;
  plan.pairs = static_cast<int>(ceil_div(rank, 128));
  int n = rows <= 32 ? 32 : 64, fixed = 0;
  for (;; n = 32) {  // 64 rows where a whole tile fits beside them, and the output in tensor memory
    fixed = 2 * plan.pairs * n * 128 + 4 * n * 128;  // Q, P
    plan.ring = (222 * 1024 - fixed) / kPairBytes;
    if ((plan.ring >= plan.pairs && (plan.pairs + 2) * 2 * n <= 512) || n == 32) break;
  }
  if (plan.ring > kMaxRing) plan.ring = kMaxRing;
  if (plan.ring < plan.pairs) return plan;
  plan.n = n;
  plan.smem = fixed + plan.ring * kPairBytes;
  plan.row_blocks = static_cast<int>(ceil_div(rows, n));
  // whole waves of CTAs, each of which costs its tiles and about five more for its start and its end
  const int64_t units = sequences * plan.row_blocks, all = ceil_div(context, static_cast<int64_t>(kTileKeys));
  int64_t best = -1;
  for (int64_t s = 1; s <= 64 && (s == 1 || 2 * s <= all); ++s) {
    const int64_t cost = ceil_div(units * s, static_cast<int64_t>(kNumSMs)) * (ceil_div(all, s) + 5);
    if (best < 0 || cost < best) {
      best = cost;
      plan.splits = static_cast<int>(s);
    }
  }
  return plan;
}

int latent_attention_tcgen05(const LatentTcPlan& plan, const void* q, const void* cache, float* partial, float2* stats,
                             const SequenceBatch& batch, int64_t rows, int64_t sequences, int64_t heads, int64_t rank,
                             int64_t slots, int64_t capacity, double scale, int32_t* status, cudaStream_t stream) {
  CUtensorMap q_map, c_map;
  if (!make_bf16_matrix_map(&q_map, q, rows * heads, rank, rank, plan.n) ||
      !make_bf16_slot_map(&c_map, cache, slots, capacity, rank, kTileKeys))
    return B200_ERR_UNSUPPORTED;
  LatentTcParams p{partial, stats, batch, status, static_cast<int>(heads), static_cast<int>(rank), plan.splits,
                   plan.pairs, plan.ring, plan.ring < 2 * plan.pairs ? 1 : 0, capacity, static_cast<float>(scale * 1.4426950408889634), wait_limit(),
                   drop_loads()};
  const dim3 grid(static_cast<unsigned>(plan.splits), static_cast<unsigned>(plan.row_blocks),
                  static_cast<unsigned>(sequences));
  auto go = [&](auto kernel) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, plan.smem) != cudaSuccess)
      return B200_ERR_LAUNCH;
    return launch_chained(kernel, grid, dim3(kThreads), plan.smem, stream, p, q_map, c_map) == cudaSuccess
               ? B200_OK : B200_ERR_LAUNCH;
  };
  return plan.n == 32 ? go(latent_attention_tcgen05_kernel<32>) : go(latent_attention_tcgen05_kernel<64>);
}

}  // namespace b200
