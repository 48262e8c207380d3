// Normalisation steps of the hybrid layers (recurrent mixers and latent attention beside each
// other, every sublayer normed before and after), all arithmetic in fp32:
//   residual_norm   x += norm_post(y); h = norm_next(x): the step between two sublayers in one
//                   launch. x is the fp32 residual stream; y the sublayer's result, in the model
//                   dtype or as fp32 split-K partial sums.
//   latent_norm     the two RMS norms behind the down projections of latent attention; the
//                   latent of every token goes straight into its cache row.
//   gated_head_norm per-head RMS norm of a recurrence's read-out, times a weight and a gate.
#include "common.cuh"
#include "hybrid.cuh"

namespace b200 {
namespace {

__device__ __forceinline__ float block_sum(float v, float* scratch) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  const int warps = (blockDim.x + 31) >> 5;
  float total = lane < warps ? scratch[lane] : 0.0f;
  total = warp_sum(total);
  __syncthreads();  // scratch is free for the next sum
  return total;
}

struct ResidualNormParams {
  float* x;             // [rows, width]: read, and written when there is a y
  const void* y;        // T [rows, y_row_stride], or fp32 partials [splits, rows, y_row_stride]; may be NULL
  const void* w_post;   // T [width]
  const void* w_next;   // T [width]; NULL: no h
  void* h;              // T [rows, h_row_stride]; columns from width on are zeroed
  int splits;           // 0: y has dtype T
  int rows, width;
  int64_t y_row_stride, h_row_stride;
  float eps, weight_offset;
};

// One CTA per row; a row's fp32 values stay in shared memory between the two norms.
template <typename T>
__global__ void __launch_bounds__(256) residual_norm_kernel(const ResidualNormParams p) {
  extern __shared__ float row_values[];
  __shared__ float scratch[32];
  grid_launch_dependents();
  grid_dependency_wait_cta();
  const int64_t row = blockIdx.x;
  float* x = p.x + row * p.width;
  float sum = 0.0f;
  if (p.y != nullptr) {
    if (p.splits > 0) {
      const float* y = static_cast<const float*>(p.y) + row * p.y_row_stride;
      const int64_t slice = static_cast<int64_t>(p.rows) * p.y_row_stride;
      for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
        const float v = sum_slices(y + c, slice, p.splits);
        row_values[c] = v;
        sum += v * v;
      }
    } else {
      const T* y = static_cast<const T*>(p.y) + row * p.y_row_stride;
      for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
        const float v = Elem<T>::load(y + c);
        row_values[c] = v;
        sum += v * v;
      }
    }
    const float factor = 1.0f / sqrtf(block_sum(sum, scratch) / p.width + p.eps);
    const T* w = static_cast<const T*>(p.w_post);
    sum = 0.0f;
    for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
      const float v = x[c] + row_values[c] * factor * (p.weight_offset + Elem<T>::load(w + c));
      x[c] = v;
      row_values[c] = v;
      sum += v * v;
    }
  } else {
    for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
      const float v = x[c];
      row_values[c] = v;
      sum += v * v;
    }
  }
  if (p.w_next == nullptr) return;
  const float factor = 1.0f / sqrtf(block_sum(sum, scratch) / p.width + p.eps);
  const T* w = static_cast<const T*>(p.w_next);
  T* h = static_cast<T*>(p.h) + row * p.h_row_stride;
  for (int c = threadIdx.x; c < p.h_row_stride; c += blockDim.x)
    Elem<T>::store(h + c, c < p.width ? row_values[c] * factor * (p.weight_offset + Elem<T>::load(w + c)) : 0.0f);
}

struct LatentNormParams {
  const void* input;  // T [rows, input_row_stride]: query latent at column 0, kv latent at kv_column
  const void* q_weight;
  const void* kv_weight;  // NULL: this layer reads another layer's latents
  void* q_out;            // T [rows, q_row_stride], zeros from q_rank on
  void* cache;            // T [slots, capacity, cache_row], zeros from kv_rank on
  void* dense;            // T [rows, cache_row] or NULL: the same rows side by side
  SequenceBatch batch;
  int rows, q_rank, kv_rank, kv_column, cache_row;
  int64_t input_row_stride, q_row_stride, capacity;
  float eps;
  int32_t* status;
};

// grid (rows, 2): y = 0 the query latent, y = 1 the kv latent
template <typename T>
__global__ void __launch_bounds__(128) latent_norm_kernel(const LatentNormParams p) {
  __shared__ float scratch[32];
  grid_launch_dependents();
  grid_dependency_wait_cta();
  const int64_t row = blockIdx.x;
  const bool kv = blockIdx.y == 1;
  const T* in = static_cast<const T*>(p.input) + row * p.input_row_stride + (kv ? p.kv_column : 0);
  const int rank = kv ? p.kv_rank : p.q_rank;
  const T* w = static_cast<const T*>(kv ? p.kv_weight : p.q_weight);
  T* out = static_cast<T*>(p.q_out) + row * p.q_row_stride;
  T* second = nullptr;
  int64_t width = p.q_row_stride;
  if (kv) {
    const int sequence = p.batch.token_sequence[row];
    const int slot = p.batch.slots[sequence];
    const int64_t position = p.batch.position(sequence, row);
    second = p.dense != nullptr ? static_cast<T*>(p.dense) + row * p.cache_row : nullptr;
    out = nullptr;
    if (slot >= 0) {
      if (position >= 0 && position < p.capacity)
        out = static_cast<T*>(p.cache) + (slot * p.capacity + position) * p.cache_row;
      else if (threadIdx.x == 0)
        atomicOr(p.status, B200_STATUS_KV_OVERFLOW);
    }
    width = p.cache_row;
  }
  float sum = 0.0f;
  for (int c = threadIdx.x; c < rank; c += blockDim.x) {
    const float v = Elem<T>::load(in + c);
    sum += v * v;
  }
  const float factor = 1.0f / sqrtf(block_sum(sum, scratch) / rank + p.eps);
  for (int64_t c = threadIdx.x; c < width; c += blockDim.x) {
    const float v = c < rank ? Elem<T>::load(in + c) * factor * Elem<T>::load(w + c) : 0.0f;
    if (out != nullptr) Elem<T>::store(out + c, v);
    if (second != nullptr) Elem<T>::store(second + c, v);
  }
}

struct GatedHeadNormParams {
  const float* input;  // [rows, heads, vdim]
  const void* weight;  // T [vdim] or NULL
  const void* gate;    // T [rows, gate_row_stride], head-major from column 0
  void* output;        // T [rows, output_row_stride], zeros from heads * vdim on
  int rows, heads, vdim, gate_kind;
  int64_t gate_row_stride, output_row_stride;
  float eps;
};

// One warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) gated_head_norm_kernel(const GatedHeadNormParams p) {
  const int lane = threadIdx.x & 31;
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  grid_launch_dependents();
  grid_dependency_wait_cta();
  if (unit >= static_cast<int64_t>(p.rows) * p.heads) return;
  const int64_t row = unit / p.heads;
  const int head = static_cast<int>(unit % p.heads);
  const float* in = p.input + unit * p.vdim;
  float sum = 0.0f;
  for (int c = lane; c < p.vdim; c += 32) sum += in[c] * in[c];
  const float factor = 1.0f / sqrtf(warp_sum(sum) / p.vdim + p.eps);
  const T* gate = static_cast<const T*>(p.gate) + row * p.gate_row_stride + static_cast<int64_t>(head) * p.vdim;
  T* out = static_cast<T*>(p.output) + row * p.output_row_stride + static_cast<int64_t>(head) * p.vdim;
  const T* w = static_cast<const T*>(p.weight);
  for (int c = lane; c < p.vdim; c += 32) {
    float v = in[c] * factor;
    if (w != nullptr) v *= Elem<T>::load(w + c);
    Elem<T>::store(out + c, v * gate_value(Elem<T>::load(gate + c), p.gate_kind));
  }
  if (head == p.heads - 1) {
    T* row_out = static_cast<T*>(p.output) + row * p.output_row_stride;
    for (int64_t c = static_cast<int64_t>(p.heads) * p.vdim + lane; c < p.output_row_stride; c += 32)
      Elem<T>::store(row_out + c, 0.0f);
  }
}

// positions[r] and the row's slot: what a replayed step reads; lengths advance behind the step
__global__ void sequence_positions_kernel(const int64_t* lengths, const int32_t* slots, int32_t* positions,
                                          int rows) {
  const int r = blockIdx.x * blockDim.x + threadIdx.x;
  if (r < rows) positions[r] = slots[r] >= 0 ? static_cast<int32_t>(lengths[slots[r]]) : 0;
}

__global__ void advance_slots_kernel(int64_t* lengths, const int32_t* slots, const int32_t* starts, int rows,
                                     int64_t capacity, int32_t* status) {
  const int r = blockIdx.x * blockDim.x + threadIdx.x;
  if (r >= rows || slots[r] < 0) return;
  const int64_t next = lengths[slots[r]] + (starts[r + 1] - starts[r]);
  if (next > capacity) atomicOr(status, B200_STATUS_KV_OVERFLOW);
  lengths[slots[r]] = next > capacity ? capacity : next;
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int b200_residual_norm(void* x, const void* y, const void* post_weight, const void* next_weight,
                                  void* h, int64_t rows, int64_t width, int64_t splits,
                                  int64_t y_row_stride, int64_t h_row_stride, double epsilon,
                                  double weight_offset, int dtype, void* stream) {
  if (!x || rows < 0 || width <= 0 || splits < 0 || (y && (!post_weight || y_row_stride < width)) ||
      (next_weight && (!h || h_row_stride < width)) || (!y && !next_weight))
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (width > 48 * 1024 || rows > INT32_MAX || splits > INT32_MAX) return B200_ERR_TOO_LARGE;
  ResidualNormParams p{static_cast<float*>(x), y, post_weight, next_weight, h, static_cast<int>(splits),
                       static_cast<int>(rows), static_cast<int>(width), y_row_stride, h_row_stride,
                       static_cast<float>(epsilon), static_cast<float>(weight_offset)};
  const size_t smem = width * sizeof(float);
  auto launch = [&](auto kernel) {
    if (smem > 48 * 1024 &&
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
      return B200_ERR_LAUNCH;
    return launch_chained(kernel, dim3(static_cast<unsigned>(rows)), dim3(256), smem,
                          static_cast<cudaStream_t>(stream), p) == cudaSuccess ? launch_status() : B200_ERR_LAUNCH;
  };
  return dtype == B200_F32 ? launch(residual_norm_kernel<float>) : launch(residual_norm_kernel<__nv_bfloat16>);
}

extern "C" int b200_latent_norm(const void* input, const void* q_weight, const void* kv_weight, void* q_out,
                                void* cache, void* dense, const int32_t* token_sequence,
                                const int32_t* starts, const int32_t* slots, const int32_t* bases,
                                int64_t rows, int64_t q_rank, int64_t kv_rank, int64_t kv_column,
                                int64_t cache_row, int64_t input_row_stride, int64_t q_row_stride,
                                int64_t capacity, double epsilon, int dtype, int32_t* status, void* stream) {
  if (!input || !q_weight || !q_out || rows < 0 || q_rank <= 0 || q_row_stride < q_rank ||
      input_row_stride < q_rank || !status)
    return B200_ERR_BAD_ARGUMENT;
  if (kv_weight && (!cache || !token_sequence || !starts || !slots || !bases || kv_rank <= 0 ||
                    cache_row < kv_rank || capacity <= 0 || kv_column < 0 || input_row_stride < kv_column + kv_rank))
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (rows > INT32_MAX) return B200_ERR_TOO_LARGE;
  LatentNormParams p{input, q_weight, kv_weight, q_out, cache, dense, {token_sequence, starts, slots, bases},
                     static_cast<int>(rows), static_cast<int>(q_rank), static_cast<int>(kv_rank),
                     static_cast<int>(kv_column), static_cast<int>(cache_row), input_row_stride, q_row_stride,
                     capacity, static_cast<float>(epsilon), status};
  const dim3 grid(static_cast<unsigned>(rows), kv_weight ? 2u : 1u);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const cudaError_t code = dtype == B200_F32 ? launch_chained(latent_norm_kernel<float>, grid, dim3(128), 0, s, p)
                                             : launch_chained(latent_norm_kernel<__nv_bfloat16>, grid, dim3(128), 0, s, p);
  return code == cudaSuccess ? launch_status() : B200_ERR_LAUNCH;
}

extern "C" int b200_gated_head_norm(const void* input, const void* weight, const void* gate, void* output,
                                    int64_t rows, int64_t heads, int64_t vdim, int64_t gate_row_stride,
                                    int64_t output_row_stride, int gate_kind, double epsilon, int dtype,
                                    void* stream) {
  if (!input || !gate || !output || rows < 0 || heads <= 0 || vdim <= 0 || gate_row_stride < heads * vdim ||
      output_row_stride < heads * vdim || (gate_kind != B200_GATE_SILU && gate_kind != B200_GATE_SIGMOID))
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (rows * heads > (static_cast<int64_t>(INT32_MAX) - 8) * 8) return B200_ERR_TOO_LARGE;
  GatedHeadNormParams p{static_cast<const float*>(input), weight, gate, output, static_cast<int>(rows),
                        static_cast<int>(heads), static_cast<int>(vdim), gate_kind, gate_row_stride,
                        output_row_stride, static_cast<float>(epsilon)};
  const dim3 grid(static_cast<unsigned>(ceil_div(rows * heads, 8)));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const cudaError_t code = dtype == B200_F32 ? launch_chained(gated_head_norm_kernel<float>, grid, dim3(256), 0, s, p)
                                             : launch_chained(gated_head_norm_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, p);
  return code == cudaSuccess ? launch_status() : B200_ERR_LAUNCH;
}

extern "C" int b200_sequence_positions(const int64_t* lengths, const int32_t* slots, int32_t* positions,
                                       int64_t rows, void* stream) {
  if (!lengths || !slots || !positions || rows < 0) return B200_ERR_BAD_ARGUMENT;
  if (rows == 0) return B200_OK;
  if (rows > INT32_MAX) return B200_ERR_TOO_LARGE;
  sequence_positions_kernel<<<static_cast<unsigned>(ceil_div(rows, 256)), 256, 0, static_cast<cudaStream_t>(stream)>>>(
      lengths, slots, positions, static_cast<int>(rows));
  return launch_status();
}

extern "C" int b200_advance_slots(int64_t* lengths, const int32_t* slots, const int32_t* starts, int64_t rows,
                                  int64_t capacity, int32_t* status, void* stream) {
  if (!lengths || !slots || !starts || !status || rows < 0 || capacity <= 0) return B200_ERR_BAD_ARGUMENT;
  if (rows == 0) return B200_OK;
  if (rows > INT32_MAX) return B200_ERR_TOO_LARGE;
  advance_slots_kernel<<<static_cast<unsigned>(ceil_div(rows, 256)), 256, 0, static_cast<cudaStream_t>(stream)>>>(
      lengths, slots, starts, static_cast<int>(rows), capacity, status);
  return launch_status();
}
