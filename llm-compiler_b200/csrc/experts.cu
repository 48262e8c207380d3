// A mixture of experts around its matrix products.
//   expert_route  sigmoid scores of the router's fp32 logits, the `top` largest of every row, and each
//                 choice's number among those of its expert (a counter per expert).
//   expert_place  the choices as rows of one matrix sorted by expert, every expert starting at a multiple of
//                 `tile` rows: the rows of h copied there, their scores, and for every tile its expert and
//                 its row count.
//   grouped_linear_generic  the product of such a matrix with a stack of weights on the CUDA cores (fp32).
// The tensor-core form is grouped_linear_tcgen05.cu. The order of rows inside an expert depends on the order
// in which counters are taken; a row's results do not depend on where it stands.
#include "common.cuh"
#include "grouped_linear.cuh"
#include "hybrid.cuh"

namespace b200 {
namespace {

// One warp per row. `top` rounds of a maximum over the logits (sigmoid grows with its argument); the lowest
// index wins ties.
__global__ void __launch_bounds__(128) expert_route_kernel(const float* logits, int32_t* chosen, float* scores,
                                                           int32_t* numbers, int32_t* counts, int64_t rows, int experts,
                                                           int top, int splits, int64_t stride) {
  extern __shared__ float values[];  // [4][experts]
  grid_launch_dependents();
  grid_dependency_wait_cta();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int64_t row = static_cast<int64_t>(blockIdx.x) * 4 + warp;
  if (row >= rows) return;
  float* own = values + warp * experts;
  for (int e = lane; e < experts; e += 32) own[e] = sum_slices(logits + row * stride + e, rows * stride, splits);
  __syncwarp();
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = INT32_MAX;
    for (int e = lane; e < experts; e += 32)
      if (own[e] > best) {
        best = own[e];
        at = e;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float other = __shfl_xor_sync(0xffffffffu, best, o);
      const int other_at = __shfl_xor_sync(0xffffffffu, at, o);
      if (other > best || (other == best && other_at < at)) {
        best = other;
        at = other_at;
      }
    }
    if (at == INT32_MAX) at = k;  // (logits that are not numbers: any expert, but a valid one)
    if (lane == 0) {
      const int64_t choice = row * top + k;
      chosen[choice] = at;
      scores[choice] = sigmoid_f32(best);
      numbers[choice] = atomicAdd(counts + at, 1);
      own[at] = -INFINITY;
    }
    __syncwarp();
  }
}

// First sorted row of every expert: a scan of the counts rounded up to whole tiles, into shared memory (the
// last entry: rows in all). Every CTA does it for itself.
__device__ __forceinline__ void scan_counts(const int32_t* counts, int experts, int tile, int* first) {
  __shared__ int warp_total[32];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  int carry = 0;
  for (int e0 = 0; e0 < experts; e0 += blockDim.x) {
    const int e = e0 + threadIdx.x;
    const int own = e < experts ? (counts[e] + tile - 1) / tile * tile : 0;
    int sum = own;
#pragma unroll
    for (int o = 1; o < 32; o *= 2) {
      const int before = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += before;
    }
    if (lane == 31) warp_total[warp] = sum;
    __syncthreads();
    int front = carry, all = carry;
    for (int w = 0; w < warps; ++w) {
      if (w < warp) front += warp_total[w];
      all += warp_total[w];
    }
    if (e < experts) first[e] = front + sum - own;
    carry = all;
    __syncthreads();
  }
  if (threadIdx.x == 0) first[experts] = carry;
  __syncthreads();
}

struct PlaceParams {
  const unsigned char* h;
  const int32_t* chosen;
  const float* scores;
  const int32_t* numbers;
  const int32_t* counts;
  int32_t* places;
  unsigned char* sorted;
  float* sorted_scores;
  int32_t* tiles;
  int64_t choices, row_bytes, h_row_bytes;
  int experts, top, tile, max_tiles;
};

// A warp per choice copies its row, 16 bytes a lane; the first CTA also writes the tile table.
__global__ void __launch_bounds__(256) expert_place_kernel(const PlaceParams p) {
  extern __shared__ int first[];  // [experts + 1]
  grid_launch_dependents();
  grid_dependency_wait_cta();
  scan_counts(p.counts, p.experts, p.tile, first);
  if (blockIdx.x == 0) {
    for (int e = threadIdx.x; e < p.experts; e += blockDim.x) {
      const int count = p.counts[e];
      for (int t = 0; t * p.tile < count; ++t) {
        const int at = first[e] / p.tile + t;
        if (at >= p.max_tiles) break;
        p.tiles[at * 2] = e;
        p.tiles[at * 2 + 1] = min(p.tile, count - t * p.tile);
      }
    }
    for (int t = first[p.experts] / p.tile + threadIdx.x; t < p.max_tiles; t += blockDim.x) {
      p.tiles[t * 2] = -1;
      p.tiles[t * 2 + 1] = 0;
    }
  }
  const int lane = threadIdx.x & 31;
  for (int64_t choice = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5); choice < p.choices;
       choice += static_cast<int64_t>(gridDim.x) * 8) {
    const int64_t place = first[p.chosen[choice]] + p.numbers[choice];
    if (place >= static_cast<int64_t>(p.max_tiles) * p.tile) {  // counters that were not zero before the routing
      if (lane == 0) p.places[choice] = 0;
      continue;
    }
    if (lane == 0) {
      p.places[choice] = static_cast<int32_t>(place);
      p.sorted_scores[place] = p.scores[choice];
    }
    const uint4* from = reinterpret_cast<const uint4*>(p.h + choice / p.top * p.h_row_bytes);
    uint4* to = reinterpret_cast<uint4*>(p.sorted + place * p.row_bytes);
    for (int64_t i = lane; i < p.row_bytes / 16; i += 32) to[i] = from[i];
  }
}

// 16 sorted rows x 64 outputs a CTA, 4 results a thread, 32 columns of K at a time.
constexpr int kRows = 16, kColumns = 64, kDepth = 32;
__global__ void __launch_bounds__(256) grouped_linear_generic_kernel(const GroupedLinearParams p, const float* x,
                                                                     const float* w) {
  __shared__ float xs[kRows][kDepth + 1], ws[kColumns][kDepth + 1];
  if (p.clear != nullptr && blockIdx.x == 0 && blockIdx.y == 0)
    for (int i = threadIdx.x; i < p.clear_count; i += blockDim.x) p.clear[i] = 0;
  const int64_t row0 = static_cast<int64_t>(blockIdx.y) * kRows;
  const int tile = static_cast<int>(row0 / p.tile), within = static_cast<int>(row0 % p.tile);
  const int expert = p.tiles[tile * 2], held = p.tiles[tile * 2 + 1] - within;
  if (expert < 0 || held <= 0) return;
  const int n0 = blockIdx.x * kColumns;
  const float* weight = w + static_cast<int64_t>(expert) * p.n * p.k;
  const int column = threadIdx.x & 63, row = (threadIdx.x >> 6) * 4;
  float acc[4] = {};
  for (int k0 = 0; k0 < p.k; k0 += kDepth) {
    for (int i = threadIdx.x; i < kRows * kDepth; i += 256) {
      const int r = i / kDepth, c = k0 + i % kDepth;
      xs[r][i % kDepth] = r < held && c < p.k ? x[(row0 + r) * p.k + c] : 0.0f;
    }
    for (int i = threadIdx.x; i < kColumns * kDepth; i += 256) {
      const int n = n0 + i / kDepth, c = k0 + i % kDepth;
      ws[i / kDepth][i % kDepth] = n < p.n && c < p.k ? weight[static_cast<int64_t>(n) * p.k + c] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < kDepth; ++c)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[i] = fmaf(xs[row + i][c], ws[column][c], acc[i]);
    __syncthreads();
  }
  float* out = static_cast<float*>(p.out);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const bool inside = row + i < held && n0 + column < p.n;
    if (p.swiglu) {
      const float s = p.scores != nullptr && row + i < held ? p.scores[row0 + row + i] : 1.0f;
      const float up = __shfl_down_sync(0xffffffffu, acc[i], 1);
      if (inside && column % 2 == 0)
        out[(row0 + row + i) * (p.n / 2) + (n0 + column) / 2] = silu_of(s * acc[i]) * (s * up);
    } else if (inside) {
      out[(row0 + row + i) * p.n + n0 + column] = acc[i];
    }
  }
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int b200_expert_route(const float* logits, int32_t* chosen, float* scores, int32_t* numbers, int32_t* counts,
                                 int64_t rows, int64_t experts, int64_t top, int64_t splits, int64_t logit_stride,
                                 void* stream) {
  if (!logits || !chosen || !scores || !numbers || !counts || rows < 0 || experts <= 0 || top <= 0 || top > experts ||
      splits <= 0 || logit_stride < experts)
    return B200_ERR_BAD_ARGUMENT;
  if (rows > INT32_MAX || rows * top > INT32_MAX || experts > 3072) return B200_ERR_TOO_LARGE;
  if (rows == 0) return B200_OK;
  const size_t smem = 4 * experts * sizeof(float);
  return launch_chained(expert_route_kernel, dim3(static_cast<unsigned>(ceil_div(rows, 4))), dim3(128), smem,
                        static_cast<cudaStream_t>(stream), logits, chosen, scores, numbers, counts, rows,
                        static_cast<int>(experts), static_cast<int>(top), static_cast<int>(splits), logit_stride) == cudaSuccess
             ? launch_status() : B200_ERR_LAUNCH;
}

extern "C" int b200_expert_place(const void* h, const int32_t* chosen, const float* scores, const int32_t* numbers,
                                 const int32_t* counts, int32_t* places, void* sorted, float* sorted_scores, int32_t* tiles,
                                 int64_t rows, int64_t experts, int64_t top, int64_t tile, int64_t max_tiles, int64_t columns,
                                 int64_t h_row_stride, int dtype, void* stream) {
  if (!h || !chosen || !scores || !numbers || !counts || !places || !sorted || !sorted_scores || !tiles || rows < 0 ||
      experts <= 0 || top <= 0 || tile <= 0 || columns <= 0 || h_row_stride < columns)
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  const int64_t element = static_cast<int64_t>(dtype_bytes(dtype));
  if (columns * element % 16 != 0 || h_row_stride * element % 16 != 0 || !aligned16(h) || !aligned16(sorted))
    return B200_ERR_ALIGNMENT;
  if (rows * top > INT32_MAX || max_tiles * tile > INT32_MAX || experts > 8192) return B200_ERR_TOO_LARGE;
  // every expert may leave a tile that is not full
  if (max_tiles < rows * top / tile + (rows * top < experts ? rows * top : experts))
    return B200_ERR_WORKSPACE;
  if (rows == 0) return B200_OK;
  PlaceParams p{static_cast<const unsigned char*>(h), chosen, scores, numbers, counts, places,
                static_cast<unsigned char*>(sorted), sorted_scores, tiles, rows * top, columns * element,
                h_row_stride * element, static_cast<int>(experts), static_cast<int>(top), static_cast<int>(tile),
                static_cast<int>(max_tiles)};
  const int64_t blocks = ceil_div(rows * top, 8);
  const dim3 grid(static_cast<unsigned>(blocks < 8 * kNumSMs ? blocks : 8 * kNumSMs));
  return launch_chained(expert_place_kernel, grid, dim3(256), (experts + 1) * sizeof(int),
                        static_cast<cudaStream_t>(stream), p) == cudaSuccess ? launch_status() : B200_ERR_LAUNCH;
}

extern "C" int b200_grouped_linear(const void* x, const void* w, const int32_t* tiles, const float* scores, void* out,
                                   int32_t* clear, int64_t clear_count, int64_t experts, int64_t tile, int64_t max_tiles,
                                   int64_t k, int64_t n, int epilogue, int dtype, int32_t* status, void* stream) {
  if (!x || !w || !tiles || !out || !status || clear_count < 0 || experts <= 0 || tile <= 0 || max_tiles < 0 || k <= 0 ||
      n <= 0 || (epilogue != B200_EPILOGUE_NONE && epilogue != B200_EPILOGUE_SWIGLU) ||
      (epilogue == B200_EPILOGUE_SWIGLU && n % 2 != 0))
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (max_tiles * tile > INT32_MAX || k > INT32_MAX || n > INT32_MAX || experts > INT32_MAX) return B200_ERR_TOO_LARGE;
  if (max_tiles == 0) return B200_OK;
  GroupedLinearParams p{tiles, scores, out, clear, status, static_cast<int>(clear_count), static_cast<int>(k),
                        static_cast<int>(n), static_cast<int>(tile), static_cast<int>(max_tiles), static_cast<int>(experts),
                        epilogue == B200_EPILOGUE_SWIGLU ? 1 : 0};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_BF16) return grouped_linear_tcgen05(p, x, w, s);
  if (tile % kRows != 0) return B200_ERR_UNSUPPORTED;
  const int64_t row_blocks = max_tiles * (tile / kRows);
  if (row_blocks > 65535) return B200_ERR_TOO_LARGE;
  const dim3 grid(static_cast<unsigned>(ceil_div(n, kColumns)), static_cast<unsigned>(row_blocks));
  grouped_linear_generic_kernel<<<grid, 256, 0, s>>>(p, static_cast<const float*>(x), static_cast<const float*>(w));
  return launch_status();
}
