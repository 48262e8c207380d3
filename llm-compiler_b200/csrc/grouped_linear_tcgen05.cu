// Products of expert-sorted rows with a stack of expert weights on tcgen05.
//
// y[r, n] = sum_k w[expert(r)][n, k] x[r, k], rows sorted by expert and padded to whole tiles. Transposed on
// the tensor core: 128 weight rows are M, the TILE sorted rows of one expert are N (16 .. 256, so that a
// decode batch with a few rows per expert pays for few), both operands K-major as they lie in memory. The
// accumulator has an output feature per TMEM lane and a row per column; the epilogue turns 32 x 32 blocks
// through shared memory into row segments.
//
// Sorted rows come in boxes of up to 64, only those that a tile holds. At decode sizes x is not sorted at all
// (index given): every item multiplies all of the step's rows, which costs the tensor core nothing beside the
// weights' stream, and the epilogue reads the columns of the rows that the tile holds.
//
// A persistent CTA per SM walks (tile, 128 features) items, features fastest: the CTAs at work at one time
// share a tile's rows, and an expert's weights are read from HBM once and from L2 by its further tiles. The
// tile table is made on the device; how many of its entries are used is known only there (the used ones come
// first). Roles: warps 0 - 3 epilogue (warp w: TMEM lanes 32 w ..), warp 4 (one lane) TMA producer into a
// ring that runs on across items, warp 5 (one lane) MMA issuer and owner of the tensor memory. Two
// accumulators: an item's epilogue runs under the next item's main loop. Every wait is bounded.
#include "common.cuh"
#include "grouped_linear.cuh"
#include "hybrid.cuh"
#include "tcgen05.cuh"
#include "tensor_map.cuh"

namespace b200 {
namespace {

constexpr int kFeatures = 128, kDepth = 64, kThreads = 192;

template <int TILE>
struct Shape {
  static constexpr int kWeightBytes = kFeatures * 128, kRowBytes = TILE * 128;
  static constexpr int kStageBytes = kWeightBytes + kRowBytes;
  static constexpr int kStages = TILE == 256 ? 4 : TILE == 128 ? 6 : 8;
  static constexpr int kColumns = TILE < 32 ? 32 : TILE;  // TMEM columns of an accumulator
  static constexpr int kStaging = 4 * 2048;               // 32 x 32 bf16 per epilogue warp
  static constexpr int kBox = TILE <= 64 ? 16 : 64;       // rows of a box of sorted rows
  static constexpr int kSmem = kStages * kStageBytes + kStaging + 1024;
};

// One column of the warp's 32 TMEM lanes, without a wait
__device__ __forceinline__ void tmem_load_column_issue(uint32_t taddr, uint32_t& r) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x1.b32 {%0}, [%1];" : "=r"(r) : "r"(taddr));
}

struct Params : GroupedLinearParams {
  uint32_t wait_limit;
  int drop_loads;
};

template <int TILE>
__global__ void __launch_bounds__(kThreads, 1)
grouped_linear_tcgen05_kernel(const Params p, const __grid_constant__ CUtensorMap w_map,
                              const __grid_constant__ CUtensorMap x_map) {
  using S = Shape<TILE>;
  constexpr int STAGES = S::kStages;
  extern __shared__ __align__(1024) unsigned char smem[];
  __shared__ __align__(8) uint64_t full_bar[STAGES], empty_bar[STAGES], acc_full[2], acc_empty[2];
  __shared__ uint32_t tmem_base_slot;
  __shared__ int failed;

  grid_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nkb = (p.k + kDepth - 1) / kDepth;
  const int features = (p.n + kFeatures - 1) / kFeatures;
  const int items = features * p.max_tiles;
  const uint32_t smem_base = smem_u32(smem);

  if (threadIdx.x == 0) {
    failed = 0;
#pragma unroll
    for (int s = 0; s < STAGES; ++s) {
      mbarrier_init(smem_u32(&full_bar[s]), 1);
      mbarrier_init(smem_u32(&empty_bar[s]), 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbarrier_init(smem_u32(&acc_full[a]), 1);
      mbarrier_init(smem_u32(&acc_empty[a]), 4);  // one arrival per epilogue warp
    }
    fence_mbarrier_init();
  }
  if (warp == 5) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;"
                 ::"r"(smem_u32(&tmem_base_slot)), "r"(static_cast<uint32_t>(2 * S::kColumns)) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem_base = tmem_base_slot;

  const int all_rows = p.index != nullptr ? p.x_rows : 0;  // 0: x is sorted

  if (warp == 4 && lane == 0 && !p.drop_loads) {
    // ---- TMA producer ----
    grid_dependency_wait();
    int round = 0;
    bool ok = true;
    for (int item = blockIdx.x; ok && item < items; item += gridDim.x) {
      const int tile = item / features, feature = (item - tile * features) * kFeatures;
      const int expert = p.tiles[tile * 2], held = min(p.tiles[tile * 2 + 1], TILE);
      if (expert < 0 || expert >= p.experts) break;
      const int first = all_rows > 0 ? 0 : tile * TILE;
      const int boxes = ((all_rows > 0 ? all_rows : held) + S::kBox - 1) / S::kBox;
      for (int kb = 0; kb < nkb; ++kb, ++round) {
        const int s = round % STAGES;
        if (round >= STAGES &&
            !mbarrier_wait_bounded(smem_u32(&empty_bar[s]), ((round / STAGES) - 1) & 1, p.wait_limit)) {
          ok = false;
          break;
        }
        const uint32_t bar = smem_u32(&full_bar[s]);
        const uint32_t w_dst = smem_base + s * S::kStageBytes;
        mbarrier_arrive_expect_tx(bar, static_cast<uint32_t>(S::kWeightBytes + boxes * S::kBox * 128));
        tma_load_3d(w_dst, &w_map, bar, kb * kDepth, feature, expert);
        for (int box = 0; box < boxes; ++box)
          tma_load_2d(w_dst + S::kWeightBytes + box * S::kBox * 128, &x_map, bar, kb * kDepth, first + box * S::kBox);
      }
    }
    if (!ok) {  // the copies still in flight get a bounded chance to land before the CTA retires
      failed = 1;
      for (int r = round < STAGES ? 0 : round - STAGES; r < round; ++r)
        mbarrier_wait_bounded(smem_u32(&full_bar[r % STAGES]), (r / STAGES) & 1, min(p.wait_limit, 100000u));
    }
  } else if (warp == 5 && lane == 0) {
    // ---- MMA issuer ----
    grid_dependency_wait();
    int round = 0, local = 0;
    bool ok = true;
    for (int item = blockIdx.x; ok && item < items; item += gridDim.x, ++local) {
      const int expert = p.tiles[item / features * 2], held = min(p.tiles[item / features * 2 + 1], TILE);
      if (expert < 0 || expert >= p.experts) break;
      const uint32_t idesc = instruction_descriptor(kFeatures, ((all_rows > 0 ? all_rows : held) + 15) / 16 * 16);
      const int acc = local & 1;
      if (local >= 2 && !mbarrier_wait_bounded(smem_u32(&acc_empty[acc]), ((local >> 1) - 1) & 1, p.wait_limit)) {
        ok = false;
        break;
      }
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t d_tmem = tmem_base + acc * S::kColumns;
      for (int kb = 0; kb < nkb; ++kb, ++round) {
        const int s = round % STAGES;
        if (!mbarrier_wait_bounded(smem_u32(&full_bar[s]), (round / STAGES) & 1, p.wait_limit)) {
          ok = false;
          break;
        }
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t w_addr = smem_base + s * S::kStageBytes;
        const uint32_t x_addr = w_addr + S::kWeightBytes;
#pragma unroll
        for (int j = 0; j < kDepth / 16; ++j)
          umma_bf16(d_tmem, smem_descriptor(w_addr + j * 32), smem_descriptor(x_addr + j * 32), idesc,
                    (kb > 0 || j > 0) ? 1u : 0u);
        umma_commit(smem_u32(&empty_bar[s]));
      }
      if (ok) umma_commit(smem_u32(&acc_full[acc]));
    }
    if (!ok) failed = 1;
  } else if (warp < 4) {
    // ---- epilogue ----
    grid_dependency_wait();
    const uint32_t staging = smem_base + STAGES * S::kStageBytes + warp * 2048;
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out);
    const int out_columns = p.swiglu ? p.n / 2 : p.n;
    int local = 0;
    bool ok = true;
    for (int item = blockIdx.x; item < items; item += gridDim.x, ++local) {
      const int tile = item / features, feature = (item - tile * features) * kFeatures;
      const int expert = p.tiles[tile * 2], held = min(p.tiles[tile * 2 + 1], TILE);
      if (expert < 0 || expert >= p.experts) break;
      const int acc = local & 1;
      // (the wait's outcome is made warp-uniform: tcgen05.ld is a warp-wide instruction)
      ok = ok && __all_sync(0xffffffffu, mbarrier_wait_bounded(smem_u32(&acc_full[acc]), (local >> 1) & 1, p.wait_limit));
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t t_addr = tmem_base + acc * S::kColumns + (static_cast<uint32_t>(warp * 32) << 16);
      const int64_t row0 = static_cast<int64_t>(tile) * TILE;
      const int own = feature + warp * 32;  // this warp's first feature
#pragma unroll 1
      for (int c0 = 0; c0 < held; c0 += 32) {
        if (own >= p.n) break;  // warp-uniform
        float v[32];
        if (all_rows > 0) {
          const int mine = p.index[row0 + min(c0 + lane, held - 1)];  // the row that stands in column c0 + lane
          uint32_t raw[32];
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int column = __shfl_sync(0xffffffffu, mine, i);
            raw[i] = 0;
            if (c0 + i < held) tmem_load_column_issue(t_addr + min(max(column, 0), all_rows - 1), raw[i]);
          }
          tmem_load_wait(raw);
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(raw[i]);
        } else {
          tmem_load_32x32(t_addr + c0, v);
        }
        __syncwarp();  // the previous block's reads of the staging tile are done
        if (p.swiglu) {
          // lanes 2 j and 2 j + 1 hold gate and up of output j: each turns one of two neighbouring rows out
          const bool is_up = lane & 1;
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const float received = __shfl_xor_sync(0xffffffffu, is_up ? v[2 * i] : v[2 * i + 1], 1);
            const int column = 2 * i + (lane & 1);
            const float s = p.scores != nullptr && c0 + column < held ? p.scores[row0 + c0 + column] : 1.0f;
            const float gate = (is_up ? received : v[2 * i]) * s, up = (is_up ? v[2 * i + 1] : received) * s;
            const float y = __fdividef(gate, 1.0f + __expf(-gate)) * up;
            asm volatile("st.shared.b16 [%0], %1;" ::"r"(staging + column * 32 + (lane >> 1) * 2),
                         "h"(f32_to_bf16_bits(y)) : "memory");
          }
          __syncwarp();
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int r = i * 16 + (lane >> 1), part = lane & 1;
            uint4 t;
            asm volatile("ld.shared.v4.b32 {%0, %1, %2, %3}, [%4];"
                         : "=r"(t.x), "=r"(t.y), "=r"(t.z), "=r"(t.w) : "r"(staging + r * 32 + part * 16));
            const int column = own / 2 + part * 8;
            if (c0 + r < held && column < out_columns)
              *reinterpret_cast<uint4*>(out + (row0 + c0 + r) * out_columns + column) = t;
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            asm volatile("st.shared.b16 [%0], %1;" ::"r"(staging + i * 64 + lane * 2), "h"(f32_to_bf16_bits(v[i])) : "memory");
          __syncwarp();
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int r = i * 8 + (lane >> 2), part = lane & 3;
            uint4 t;
            asm volatile("ld.shared.v4.b32 {%0, %1, %2, %3}, [%4];"
                         : "=r"(t.x), "=r"(t.y), "=r"(t.z), "=r"(t.w) : "r"(staging + r * 64 + part * 16));
            const int column = own + part * 8;
            if (c0 + r < held && column < out_columns)
              *reinterpret_cast<uint4*>(out + (row0 + c0 + r) * out_columns + column) = t;
          }
        }
      }
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0)
        asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&acc_empty[acc])) : "memory");
    }
    if (!ok) failed = 1;
  }
  __syncwarp();
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (failed && threadIdx.x == 0) atomicOr(p.status, B200_STATUS_WAIT_TIMEOUT);
  if (warp == 5)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base),
                 "r"(static_cast<uint32_t>(2 * S::kColumns)) : "memory");
}

template <int TILE>
int launch(const Params& p, const CUtensorMap& w_map, const CUtensorMap& x_map, cudaStream_t stream) {
  static_assert(Shape<TILE>::kSmem <= 227 * 1024, "stage ring exceeds shared memory");
  auto kernel = grouped_linear_tcgen05_kernel<TILE>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, Shape<TILE>::kSmem) != cudaSuccess)
    return B200_ERR_LAUNCH;
  const int64_t items = ceil_div(p.n, kFeatures) * p.max_tiles;
  const dim3 grid(static_cast<unsigned>(items < kNumSMs ? items : kNumSMs));
  if (launch_chained(kernel, grid, dim3(kThreads), Shape<TILE>::kSmem, stream, p, w_map, x_map) != cudaSuccess)
    return B200_ERR_LAUNCH;
  return launch_status();
}

}  // namespace

int grouped_linear_tcgen05(const GroupedLinearParams& in, const void* x, const void* w, cudaStream_t stream) {
  if (in.index != nullptr && in.x_rows > in.tile) return B200_ERR_UNSUPPORTED;
  if (in.k % 8 != 0 || in.n % (in.swiglu ? 16 : 8) != 0) return B200_ERR_UNSUPPORTED;
  if (!aligned16(x) || !aligned16(w) || !aligned16(in.out)) return B200_ERR_ALIGNMENT;
  if (ceil_div(in.n, kFeatures) * in.max_tiles > INT32_MAX) return B200_ERR_TOO_LARGE;
  CUtensorMap w_map, x_map;
  if (!make_bf16_slot_map(&w_map, w, in.experts, in.n, in.k, kFeatures) ||
      !make_bf16_matrix_map(&x_map, x, in.x_rows, in.k, in.k, in.tile <= 64 ? 16 : 64))
    return B200_ERR_UNSUPPORTED;
  Params p;
  static_cast<GroupedLinearParams&>(p) = in;
  p.wait_limit = wait_limit();
  p.drop_loads = drop_loads();
  switch (in.tile) {
    case 16: return launch<16>(p, w_map, x_map, stream);
    case 32: return launch<32>(p, w_map, x_map, stream);
    case 64: return launch<64>(p, w_map, x_map, stream);
    case 128: return launch<128>(p, w_map, x_map, stream);
    case 256: return launch<256>(p, w_map, x_map, stream);
    default: return B200_ERR_UNSUPPORTED;
  }
}

}  // namespace b200
