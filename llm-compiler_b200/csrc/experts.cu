// A mixture of experts around its matrix products: which rows go to which expert, with what score.
//
// Every row takes the `top` experts with the largest router logits (sigmoid scores grow with them). The
// choices become rows of an expert-sorted order in which every expert starts at a multiple of `tile` rows:
// index[sorted row] is the row of h, sorted_scores its score, tiles[t] the expert of a tile and how many of
// its rows are held, places[row] the sorted rows that belong to a row of h. `always` more experts, numbered
// from `experts` on, take every row with score 1 and stand in front.
//   expert_select  decode sizes: router products, choice and order in one launch, a CTA per row; the CTA
//                  that finishes last puts the choices in order.
//   expert_route, expert_place  prompts: choice from finished logits, then the order and the rows in it.
//   grouped_linear_generic  the product of sorted rows with a stack of weights on the CUDA cores (fp32); the
//                  tensor-core form is grouped_linear_tcgen05.cu.
// The order of rows inside an expert depends on the order in which counters are taken; a row's results do not
// depend on where it stands.
#include "common.cuh"
#include "grouped_linear.cuh"
#include "hybrid.cuh"

namespace b200 {
namespace {

struct OrderParams {
  const int32_t* chosen;   // [rows, top]
  const float* scores;     // [rows, top]
  int32_t* numbers;        // [rows, top]: a choice's number among its expert's
  int32_t* counters;       // [experts] rows of every expert, then a ticket; zero between calls
  int32_t* places;         // [rows, always + top]
  int32_t* index;          // [max_tiles * tile]
  float* sorted_scores;    // [max_tiles * tile]
  int32_t* tiles;          // [max_tiles][2]
  int64_t rows;
  int experts, top, always, tile, max_tiles;
};

// Warp-wide: the `top` largest of values [experts] (overwritten), lowest index first among equals.
// take(k, expert, value) runs on lane 0.
template <typename Take>
__device__ __forceinline__ void choose_largest(float* values, int experts, int top, int lane, Take take) {
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = INT32_MAX;
    for (int e = lane; e < experts; e += 32)
      if (values[e] > best) {
        best = values[e];
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
      take(k, at, best);
      values[at] = -INFINITY;
    }
    __syncwarp();
  }
}

// First sorted row of every expert (behind those that take every row), into shared memory; the last entry:
// rows in all. Every CTA does it for itself.
template <typename Count>
__device__ __forceinline__ void scan_counts(const OrderParams& p, int* first, Count count) {
  __shared__ int warp_total[32];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  int carry = p.always * static_cast<int>((p.rows + p.tile - 1) / p.tile) * p.tile;
  for (int e0 = 0; e0 < p.experts; e0 += blockDim.x) {
    const int e = e0 + threadIdx.x;
    const int own = e < p.experts ? (count(e) + p.tile - 1) / p.tile * p.tile : 0;
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
    if (e < p.experts) first[e] = front + sum - own;
    carry = all;
    __syncthreads();
  }
  if (threadIdx.x == 0) first[p.experts] = carry;
  __syncthreads();
}

template <typename Count>
__device__ __forceinline__ void write_tiles(const OrderParams& p, const int* first, Count count_of) {
  const int whole = static_cast<int>((p.rows + p.tile - 1) / p.tile);  // tiles of an expert that takes every row
  for (int t = threadIdx.x; t < p.always * whole; t += blockDim.x) {
    const int64_t left = p.rows - static_cast<int64_t>(t % whole) * p.tile;
    p.tiles[t * 2] = p.experts + t / whole;
    p.tiles[t * 2 + 1] = left < p.tile ? static_cast<int>(left) : p.tile;
  }
  for (int e = threadIdx.x; e < p.experts; e += blockDim.x) {
    const int count = count_of(e);
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

// Sorted row `place` belongs to `row` as its k-th of always + top
__device__ __forceinline__ bool write_choice(const OrderParams& p, int64_t row, int k, int64_t place, float score) {
  // (counters that were not zero before the call would lead outside)
  const bool inside = place < static_cast<int64_t>(p.max_tiles) * p.tile;
  p.places[row * (p.always + p.top) + k] = inside ? static_cast<int32_t>(place) : 0;
  if (inside) {
    p.index[place] = static_cast<int32_t>(row);
    p.sorted_scores[place] = score;
  }
  return inside;
}

// The CTA that arrives last at the ticket (every thread gets the answer). Thread 0 publishes what it has
// written itself.
__device__ __forceinline__ bool arrive_last(int32_t* ticket) {
  __shared__ int last;
  if (threadIdx.x == 0) __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) last = atomicAdd(ticket, 1) == static_cast<int>(gridDim.x) - 1;
  __syncthreads();
  if (last) __threadfence();
  return last != 0;
}

// A CTA per row. The products with the router are fp32 sums of exact products of the operands.
template <typename T>
__global__ void __launch_bounds__(512) expert_select_kernel(const OrderParams p, const T* h, const T* router, int width,
                                                            int64_t h_stride, int32_t* chosen, float* scores,
                                                            int early_weights) {
  extern __shared__ float logits[];  // [experts], then first rows [experts + 1], counts [experts]
  constexpr int V = Elem<T>::kPerVec;
  int* first = reinterpret_cast<int*>(logits + p.experts);
  int* counts = first + p.experts + 1;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  grid_launch_dependents();
  if (early_weights) {  // the router's weights are constants: this CTA's share of them into L2 before the wait
    const int64_t lines = static_cast<int64_t>(p.experts) * width * static_cast<int>(sizeof(T)) / 128;
    for (int64_t i = blockIdx.x + static_cast<int64_t>(threadIdx.x) * gridDim.x; i < lines; i += static_cast<int64_t>(blockDim.x) * gridDim.x)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(router) + i * 128));
  }
  grid_dependency_wait_cta();
  const T* row = h + blockIdx.x * h_stride;
  for (int e0 = warp * 2; e0 < p.experts; e0 += warps * 2) {  // two experts a warp: twice the loads in flight
    const int e1 = e0 + 1 < p.experts ? e0 + 1 : e0;
    float a = 0.0f, b = 0.0f;
#pragma unroll 4
    for (int c = lane * V; c < width; c += 32 * V) {
      Vec16<T> x, ta, tb;
      x.load(row + c);
      ta.load(router + static_cast<int64_t>(e0) * width + c);
      tb.load(router + static_cast<int64_t>(e1) * width + c);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        a = fmaf(ta.v[i], x.v[i], a);
        b = fmaf(tb.v[i], x.v[i], b);
      }
    }
    a = warp_sum(a);
    b = warp_sum(b);
    if (lane == 0) {
      logits[e0] = a;
      if (e1 > e0) logits[e1] = b;
    }
  }
  for (int e = threadIdx.x; e < p.experts; e += blockDim.x) counts[e] = 0;
  __syncthreads();
  if (warp == 0)
    choose_largest(logits, p.experts, p.top, lane, [&](int k, int expert, float logit) {
      const int64_t choice = static_cast<int64_t>(blockIdx.x) * p.top + k;
      chosen[choice] = expert;
      scores[choice] = sigmoid_f32(logit);
    });
  if (!arrive_last(p.counters + p.experts)) return;
  // ---- the order: numbers from counters in shared memory, kept in p.numbers between the two passes ----
  const int choices = static_cast<int>(p.rows) * p.top;
  constexpr int kKept = 4;  // choices a thread remembers
  int expert_of[kKept], number_of[kKept];
#pragma unroll
  for (int j = 0; j < kKept; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    expert_of[j] = i < choices ? __ldcg(chosen + i) : 0;
  }
#pragma unroll
  for (int j = 0; j < kKept; ++j)
    number_of[j] = threadIdx.x + j * static_cast<int>(blockDim.x) < choices ? atomicAdd(counts + expert_of[j], 1) : 0;
  for (int i = threadIdx.x + kKept * blockDim.x; i < choices; i += blockDim.x)
    p.numbers[i] = atomicAdd(counts + __ldcg(chosen + i), 1);
  __syncthreads();
  auto count = [&](int e) { return counts[e]; };
  scan_counts(p, first, count);
  write_tiles(p, first, count);
#pragma unroll
  for (int j = 0; j < kKept; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < choices) write_choice(p, i / p.top, p.always + i % p.top, first[expert_of[j]] + number_of[j], __ldcg(scores + i));
  }
  for (int i = threadIdx.x + kKept * blockDim.x; i < choices; i += blockDim.x)
    write_choice(p, i / p.top, p.always + i % p.top, first[__ldcg(chosen + i)] + p.numbers[i], __ldcg(scores + i));
  const int whole = static_cast<int>((p.rows + p.tile - 1) / p.tile) * p.tile;
  for (int i = threadIdx.x; i < p.always * static_cast<int>(p.rows); i += blockDim.x) {
    const int k = i / static_cast<int>(p.rows), r = i - k * static_cast<int>(p.rows);
    write_choice(p, r, k, k * static_cast<int64_t>(whole) + r, 1.0f);
  }
  if (threadIdx.x == 0) p.counters[p.experts] = 0;
}

// 32 rows a CTA, four a warp; numbers are taken from the CTA's own counts, then from the global ones at once.
constexpr int kRouteRows = 32;
__global__ void __launch_bounds__(256) expert_route_kernel(const float* logits, int32_t* chosen, float* scores,
                                                           int32_t* numbers, int32_t* counters, int64_t rows, int experts,
                                                           int top, int splits, int64_t stride) {
  extern __shared__ float values[];  // [8][experts], then counts [experts], choices and numbers [32 * top] each
  int* counts = reinterpret_cast<int*>(values + 8 * experts);
  int* own_chosen = counts + experts;
  int* own_numbers = own_chosen + kRouteRows * top;
  grid_launch_dependents();
  grid_dependency_wait_cta();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int e = threadIdx.x; e < experts; e += blockDim.x) counts[e] = 0;
  __syncthreads();
  const int64_t row0 = static_cast<int64_t>(blockIdx.x) * kRouteRows;
  float* own = values + warp * experts;
  for (int r = warp; r < kRouteRows && row0 + r < rows; r += 8) {
    for (int e = lane; e < experts; e += 32) own[e] = sum_slices(logits + (row0 + r) * stride + e, rows * stride, splits);
    __syncwarp();
    choose_largest(own, experts, top, lane, [&](int k, int expert, float logit) {
      own_chosen[r * top + k] = expert;
      own_numbers[r * top + k] = atomicAdd(counts + expert, 1);
      scores[(row0 + r) * top + k] = sigmoid_f32(logit);
    });
  }
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += blockDim.x)
    if (counts[e] > 0) counts[e] = atomicAdd(counters + e, counts[e]);
  __syncthreads();
  for (int i = threadIdx.x; i < kRouteRows * top && row0 * top + i < rows * top; i += blockDim.x) {
    chosen[row0 * top + i] = own_chosen[i];
    numbers[row0 * top + i] = counts[own_chosen[i]] + own_numbers[i];
  }
}

// A warp per choice: its place, and its row of h copied there, 16 bytes a lane.
__global__ void __launch_bounds__(256) expert_place_kernel(const OrderParams p, const unsigned char* h, unsigned char* sorted,
                                                           int64_t row_bytes, int64_t h_row_bytes) {
  extern __shared__ int first[];  // [experts + 1]
  grid_launch_dependents();
  grid_dependency_wait_cta();
  auto count = [&](int e) { return __ldcg(p.counters + e); };
  scan_counts(p, first, count);
  if (blockIdx.x == 0) write_tiles(p, first, count);
  const int lane = threadIdx.x & 31, each = p.always + p.top;
  const int64_t whole = (p.rows + p.tile - 1) / p.tile * p.tile;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5); i < p.rows * each; i += static_cast<int64_t>(gridDim.x) * 8) {
    const int64_t row = i / each;
    const int k = static_cast<int>(i - row * each);
    const int64_t choice = row * p.top + k - p.always;
    const int64_t place = k < p.always ? k * whole + row : first[p.chosen[choice]] + p.numbers[choice];
    bool inside = false;
    if (lane == 0) inside = write_choice(p, row, k, place, k < p.always ? 1.0f : p.scores[choice]);
    inside = __shfl_sync(0xffffffffu, inside ? 1 : 0, 0) != 0;
    if (h == nullptr || !inside) continue;
    const uint4* from = reinterpret_cast<const uint4*>(h + row * h_row_bytes);
    uint4* to = reinterpret_cast<uint4*>(sorted + place * row_bytes);
    const int64_t units = row_bytes / 16;
    for (int64_t u = lane; u < units; u += 128) {
      uint4 t[4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (u + 32 * j < units) t[j] = from[u + 32 * j];
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (u + 32 * j < units) to[u + 32 * j] = t[j];
    }
  }
  if (!arrive_last(p.counters + p.experts)) return;  // (every CTA has read the counters)
  for (int e = threadIdx.x; e <= p.experts; e += blockDim.x) p.counters[e] = 0;
}

// 16 sorted rows x 64 outputs a CTA, 4 results a thread, 32 columns of K at a time.
constexpr int kRows = 16, kColumns = 64, kDepth = 32;
__global__ void __launch_bounds__(256) grouped_linear_generic_kernel(const GroupedLinearParams p, const float* x,
                                                                     const float* w) {
  __shared__ float xs[kRows][kDepth + 1], ws[kColumns][kDepth + 1];
  const int64_t row0 = static_cast<int64_t>(blockIdx.y) * kRows;
  const int tile = static_cast<int>(row0 / p.tile), within = static_cast<int>(row0 % p.tile);
  const int expert = p.tiles[tile * 2], held = p.tiles[tile * 2 + 1] - within;
  if (expert < 0 || expert >= p.experts || held <= 0) return;
  const int n0 = blockIdx.x * kColumns;
  const float* weight = w + static_cast<int64_t>(expert) * p.n * p.k;
  const int column = threadIdx.x & 63, row = (threadIdx.x >> 6) * 4;
  float acc[4] = {};
  for (int k0 = 0; k0 < p.k; k0 += kDepth) {
    for (int i = threadIdx.x; i < kRows * kDepth; i += 256) {
      const int r = i / kDepth, c = k0 + i % kDepth;
      float v = 0.0f;
      if (r < held && c < p.k) v = x[(p.index != nullptr ? p.index[row0 + r] : row0 + r) * p.k + c];
      xs[r][i % kDepth] = v;
    }
    for (int i = threadIdx.x; i < kColumns * kDepth; i += 256) {
      const int n = n0 + i / kDepth, c = k0 + i % kDepth;
      ws[i / kDepth][i % kDepth] = n < p.n && c < p.k ? weight[static_cast<int64_t>(n) * p.k + c] : 0.0f;
    }
    __syncthreads();
    float block[4] = {};
#pragma unroll
    for (int c = 0; c < kDepth; ++c)
#pragma unroll
      for (int i = 0; i < 4; ++i) block[i] = fmaf(xs[row + i][c], ws[column][c], block[i]);
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[i] += block[i];
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

int order_params(const b200_expert_order* in, int64_t rows, OrderParams* out) {
  if (in == nullptr || !in->chosen || !in->scores || !in->numbers || !in->counters || !in->places || !in->index ||
      !in->sorted_scores || !in->tiles || rows < 0 || in->experts <= 0 || in->top <= 0 || in->top > in->experts ||
      in->always < 0 || in->tile <= 0)
    return B200_ERR_BAD_ARGUMENT;
  if (rows * (in->top + in->always) > INT32_MAX || in->max_tiles * in->tile > INT32_MAX || in->experts > 4096 ||
      in->always > 4096)
    return B200_ERR_TOO_LARGE;
  const int64_t choices = rows * in->top;  // every expert may leave a tile that is not full
  if (in->max_tiles < in->always * ceil_div(rows, in->tile) + choices / in->tile + (choices < in->experts ? choices : in->experts))
    return B200_ERR_WORKSPACE;
  *out = OrderParams{in->chosen, in->scores, in->numbers, in->counters, in->places, in->index, in->sorted_scores, in->tiles,
                     rows, static_cast<int>(in->experts), static_cast<int>(in->top), static_cast<int>(in->always),
                     static_cast<int>(in->tile), static_cast<int>(in->max_tiles)};
  return B200_OK;
}

template <typename Kernel>
bool allow_shared(Kernel kernel, size_t smem) {
  return smem <= 48 * 1024 ||
         cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) == cudaSuccess;
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int b200_expert_select(const void* h, const void* router, const b200_expert_order* order, int64_t rows,
                                  int64_t width, int64_t h_row_stride, int dtype, void* stream) {
  OrderParams p;
  const int code = order_params(order, rows, &p);
  if (code != B200_OK) return code;
  if (!h || !router || width <= 0 || h_row_stride < width) return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (width % 8 != 0 || h_row_stride % 8 != 0 || !aligned16(h) || !aligned16(router)) return B200_ERR_ALIGNMENT;
  if (rows == 0) return B200_OK;
  const size_t smem = (3 * p.experts + 1) * sizeof(float);
  if (rows > 65535 || smem > 200 * 1024) return B200_ERR_TOO_LARGE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto go = [&](auto tag) {
    using T = typename decltype(tag)::type;
    auto kernel = expert_select_kernel<T>;
    return allow_shared(kernel, smem) &&
                   launch_chained(kernel, dim3(static_cast<unsigned>(rows)), dim3(p.experts > 16 ? 512 : 256), smem, s, p,
                                  static_cast<const T*>(h), static_cast<const T*>(router), static_cast<int>(width),
                                  h_row_stride, order->chosen, order->scores,
                                  (launch_mode() & B200_LAUNCH_CONSTANT_WEIGHTS) != 0 ? 1 : 0) == cudaSuccess
               ? launch_status() : B200_ERR_LAUNCH;
  };
  return dtype == B200_F32 ? go(TypeTag<float>{}) : go(TypeTag<__nv_bfloat16>{});
}

extern "C" int b200_expert_route(const float* logits, const b200_expert_order* order, int64_t rows, int64_t splits,
                                 int64_t logit_stride, void* stream) {
  OrderParams p;
  const int code = order_params(order, rows, &p);
  if (code != B200_OK) return code;
  if (!logits || splits <= 0 || splits > INT32_MAX || logit_stride < p.experts) return B200_ERR_BAD_ARGUMENT;
  if (rows == 0) return B200_OK;
  const size_t smem = (9 * p.experts + 2 * kRouteRows * p.top) * sizeof(float);
  const int64_t blocks = ceil_div(rows, kRouteRows);
  if (smem > 200 * 1024 || blocks > INT32_MAX) return B200_ERR_TOO_LARGE;
  return allow_shared(expert_route_kernel, smem) &&
                 launch_chained(expert_route_kernel, dim3(static_cast<unsigned>(blocks)), dim3(256), smem,
                                static_cast<cudaStream_t>(stream), logits, order->chosen, order->scores, order->numbers,
                                order->counters, rows, p.experts, p.top, static_cast<int>(splits), logit_stride) == cudaSuccess
             ? launch_status() : B200_ERR_LAUNCH;
}

extern "C" int b200_expert_place(const b200_expert_order* order, const void* h, void* sorted, int64_t rows,
                                 int64_t columns, int64_t h_row_stride, int dtype, void* stream) {
  OrderParams p;
  const int code = order_params(order, rows, &p);
  if (code != B200_OK) return code;
  if (h != nullptr && (!sorted || columns <= 0 || h_row_stride < columns)) return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  const int64_t element = static_cast<int64_t>(dtype_bytes(dtype));
  if (h != nullptr && (columns * element % 16 != 0 || h_row_stride * element % 16 != 0 || !aligned16(h) || !aligned16(sorted)))
    return B200_ERR_ALIGNMENT;
  if (rows == 0) return B200_OK;
  const int64_t blocks = ceil_div(rows * (p.top + p.always), 8);
  return launch_chained(expert_place_kernel, dim3(static_cast<unsigned>(blocks < 8 * kNumSMs ? blocks : 8 * kNumSMs)),
                        dim3(256), (p.experts + 1) * sizeof(int), static_cast<cudaStream_t>(stream), p,
                        static_cast<const unsigned char*>(h), static_cast<unsigned char*>(sorted), columns * element,
                        h_row_stride * element) == cudaSuccess
             ? launch_status() : B200_ERR_LAUNCH;
}

extern "C" int b200_grouped_linear(const void* x, const void* w, const int32_t* tiles, const int32_t* index,
                                   const float* scores, void* out, int64_t experts, int64_t tile, int64_t max_tiles,
                                   int64_t x_rows, int64_t k, int64_t n, int epilogue, int dtype, int32_t* status,
                                   void* stream) {
  if (!x || !w || !tiles || !out || !status || experts <= 0 || tile <= 0 || max_tiles < 0 || k <= 0 || n <= 0 ||
      x_rows < 0 || (!index && x_rows < max_tiles * tile) ||
      (epilogue != B200_EPILOGUE_NONE && epilogue != B200_EPILOGUE_SWIGLU) || (epilogue == B200_EPILOGUE_SWIGLU && n % 2 != 0))
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (max_tiles * tile > INT32_MAX || x_rows > INT32_MAX || k > INT32_MAX || n > INT32_MAX || experts > INT32_MAX)
    return B200_ERR_TOO_LARGE;
  if (max_tiles == 0 || x_rows == 0) return B200_OK;
  GroupedLinearParams p{tiles, index, scores, out, status, static_cast<int>(k), static_cast<int>(n), static_cast<int>(tile),
                        static_cast<int>(max_tiles), static_cast<int>(x_rows), static_cast<int>(experts),
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
