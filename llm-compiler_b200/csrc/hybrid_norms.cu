// Normalisation steps of the hybrid layers (recurrent mixers and attention beside each other, a norm
// behind every sublayer, in some designs one in front of it as well), all arithmetic in fp32:
//   residual_norm   x += norm_post(y); h = norm_next(x), or x itself: the step between two sublayers
//                   in one launch. x is the fp32 residual stream; y the sublayer's result, in the model
//                   dtype or as fp32 split-K partial sums, plus the rows that a token's experts left.
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
  const void* w_next;   // T [width]; NULL: h is x itself, without a norm
  void* h;              // T [rows, h_row_stride]; columns from width on are zeroed; NULL: no h
  int splits;           // 0: y has dtype T
  int rows, width;
  int64_t y_row_stride, h_row_stride;
  float eps, weight_offset;
  // y also takes the sum of rows places[row, 0 .. top - 1] of this matrix (top 0: none)
  const void* summands; // T [any, summand_row_stride]
  const int32_t* places;
  int top;
  int64_t summand_row_stride;
  const void* y_bias;   // T [width] added to every y, or NULL
  __device__ __forceinline__ bool adds() const { return y != nullptr || top > 0; }
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
  if (p.adds()) {
    const int64_t slice = static_cast<int64_t>(p.rows) * p.y_row_stride;
    for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
      float v = 0.0f;
      if (p.y != nullptr)
        v = p.splits > 0 ? sum_slices(static_cast<const float*>(p.y) + row * p.y_row_stride + c, slice, p.splits)
                         : Elem<T>::load(static_cast<const T*>(p.y) + row * p.y_row_stride + c);
      if (p.y_bias != nullptr) v += Elem<T>::load(static_cast<const T*>(p.y_bias) + c);
      for (int k = 0; k < p.top; ++k)
        v += Elem<T>::load(static_cast<const T*>(p.summands) + p.places[row * p.top + k] * p.summand_row_stride + c);
      row_values[c] = v;
      sum += v * v;
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
  if (p.h == nullptr) return;
  T* h = static_cast<T*>(p.h) + row * p.h_row_stride;
  const T* w = static_cast<const T*>(p.w_next);
  if (w == nullptr) {
    for (int c = threadIdx.x; c < p.h_row_stride; c += blockDim.x) Elem<T>::store(h + c, c < p.width ? row_values[c] : 0.0f);
    return;
  }
  const float factor = 1.0f / sqrtf(block_sum(sum, scratch) / p.width + p.eps);
  for (int c = threadIdx.x; c < p.h_row_stride; c += blockDim.x)
    Elem<T>::store(h + c, c < p.width ? row_values[c] * factor * (p.weight_offset + Elem<T>::load(w + c)) : 0.0f);
}

// Four elements of a model-dtype row
template <typename T>
__device__ __forceinline__ float4 load_quad(const T* p) {
  if (sizeof(T) == 4) return *reinterpret_cast<const float4*>(p);
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y));
}
template <typename T>
__device__ __forceinline__ void store_quad(T* p, float4 v) {
  if (sizeof(T) == 4) *reinterpret_cast<float4*>(p) = v;
  else *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ float squares_of(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// The same for widths that are a multiple of four: four columns an access, the row in registers, every
// load of the row in flight at once.
template <typename T, int Q>
__global__ void __launch_bounds__(Q == 1 ? 1024 : 512) residual_norm_quads_kernel(const ResidualNormParams p) {
  __shared__ float scratch[32];
  grid_launch_dependents();
  const int quads = p.width / 4;
  const int64_t row = blockIdx.x;
  float* x = p.x + row * p.width;
  const T* post = static_cast<const T*>(p.w_post);
  const T* next = static_cast<const T*>(p.w_next);
  grid_dependency_wait_cta();
  float4 v[Q], y[Q];
  float sum = 0.0f;
#pragma unroll
  for (int i = 0; i < Q; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    v[i] = c < quads ? *reinterpret_cast<const float4*>(x + c * 4) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  if (p.adds()) {
#pragma unroll
    for (int i = 0; i < Q; ++i) y[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (p.y != nullptr && p.splits > 0) {
      const float* partial = static_cast<const float*>(p.y) + row * p.y_row_stride;
      const int64_t slice = static_cast<int64_t>(p.rows) * p.y_row_stride;
#pragma unroll
      for (int i = 0; i < Q; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c >= quads) continue;
        for (int s0 = 0; s0 < p.splits; s0 += 4) {
          float4 t[4];
#pragma unroll
          for (int s = 0; s < 4; ++s)
            t[s] = s0 + s < p.splits ? __ldcg(reinterpret_cast<const float4*>(partial + (s0 + s) * slice + c * 4))
                                     : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
          for (int s = 0; s < 4; ++s) {
            y[i].x += t[s].x; y[i].y += t[s].y; y[i].z += t[s].z; y[i].w += t[s].w;
          }
        }
      }
    } else if (p.y != nullptr) {
      const T* in = static_cast<const T*>(p.y) + row * p.y_row_stride;
#pragma unroll
      for (int i = 0; i < Q; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < quads) y[i] = load_quad<T>(in + c * 4);
      }
    }
    if (p.y_bias != nullptr) {
#pragma unroll
      for (int i = 0; i < Q; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c >= quads) continue;
        const float4 t = load_quad<T>(static_cast<const T*>(p.y_bias) + c * 4);
        y[i].x += t.x; y[i].y += t.y; y[i].z += t.z; y[i].w += t.w;
      }
    }
#pragma unroll 2
    for (int k = 0; k < p.top; ++k) {
      const T* in = static_cast<const T*>(p.summands) + p.places[row * p.top + k] * p.summand_row_stride;
#pragma unroll
      for (int i = 0; i < Q; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c >= quads) continue;
        const float4 t = load_quad<T>(in + c * 4);
        y[i].x += t.x; y[i].y += t.y; y[i].z += t.z; y[i].w += t.w;
      }
    }
#pragma unroll
    for (int i = 0; i < Q; ++i) sum += squares_of(y[i]);
    const float factor = 1.0f / sqrtf(block_sum(sum, scratch) / p.width + p.eps);
#pragma unroll
    for (int i = 0; i < Q; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c >= quads) continue;
      const float4 w = load_quad<T>(post + c * 4);
      v[i].x += y[i].x * factor * (p.weight_offset + w.x);
      v[i].y += y[i].y * factor * (p.weight_offset + w.y);
      v[i].z += y[i].z * factor * (p.weight_offset + w.z);
      v[i].w += y[i].w * factor * (p.weight_offset + w.w);
      *reinterpret_cast<float4*>(x + c * 4) = v[i];
    }
  }
  if (p.h == nullptr) return;
  T* h = static_cast<T*>(p.h) + row * p.h_row_stride;
  if (static_cast<int>(threadIdx.x) < p.h_row_stride - p.width) Elem<T>::store(h + p.width + threadIdx.x, 0.0f);
  if (p.w_next == nullptr) {
#pragma unroll
    for (int i = 0; i < Q; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < quads) store_quad<T>(h + c * 4, v[i]);
    }
    return;
  }
  sum = 0.0f;
#pragma unroll
  for (int i = 0; i < Q; ++i) sum += squares_of(v[i]);
  const float factor = 1.0f / sqrtf(block_sum(sum, scratch) / p.width + p.eps);
#pragma unroll
  for (int i = 0; i < Q; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    if (c >= quads) continue;
    const float4 w = load_quad<T>(next + c * 4);
    store_quad<T>(h + c * 4, make_float4(v[i].x * factor * (p.weight_offset + w.x), v[i].y * factor * (p.weight_offset + w.y),
                                         v[i].z * factor * (p.weight_offset + w.z), v[i].w * factor * (p.weight_offset + w.w)));
  }
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

// The same for vdim 64 or 128 (V) and 16-byte rows: V / 4 lanes a (row, head), four columns each.
template <typename T, int V>
__global__ void __launch_bounds__(256) gated_head_norm_quads_kernel(const GatedHeadNormParams p) {
  constexpr int L = V / 4;
  grid_launch_dependents();
  grid_dependency_wait_cta();
  const int64_t unit = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) / L;
  const bool inside = unit < static_cast<int64_t>(p.rows) * p.heads;
  const int64_t row = inside ? unit / p.heads : 0;
  const int head = inside ? static_cast<int>(unit - row * p.heads) : 0, c = threadIdx.x % L * 4;
  const int64_t at = static_cast<int64_t>(head) * V + c;
  float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f), gate = v;
  if (inside) {
    v = __ldcs(reinterpret_cast<const float4*>(p.input + unit * V + c));
    gate = load_quad<T>(static_cast<const T*>(p.gate) + row * p.gate_row_stride + at);
  }
  float sum = squares_of(v);
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  if (!inside) return;
  const float factor = 1.0f / sqrtf(sum / V + p.eps);
  const float4 w = p.weight != nullptr ? load_quad<T>(static_cast<const T*>(p.weight) + c) : make_float4(1.0f, 1.0f, 1.0f, 1.0f);
  store_quad<T>(static_cast<T*>(p.output) + row * p.output_row_stride + at,
                make_float4(v.x * factor * w.x * gate_value(gate.x, p.gate_kind), v.y * factor * w.y * gate_value(gate.y, p.gate_kind),
                            v.z * factor * w.z * gate_value(gate.z, p.gate_kind), v.w * factor * w.w * gate_value(gate.w, p.gate_kind)));
}

// The residual stream's first rows: a row of the table per id, widened to fp32; with `weight` normed (RMS,
// times weight_offset + weight), and with `h` also in the model dtype.
struct EmbeddingParams {
  const void* table;  // T [vocab, width]
  const void* weight; // T [width] or NULL
  const int64_t* ids;
  float* x;           // [rows, width]
  void* h;            // T [rows, h_row_stride] or NULL, zeros from width on
  int width;
  int64_t vocab, h_row_stride;
  float eps, weight_offset;
  int32_t* status;
};
template <typename T>
__global__ void __launch_bounds__(256) embedding_residual_kernel(const EmbeddingParams p) {
  __shared__ float scratch[32];
  const int64_t row = blockIdx.x, id = p.ids[row];
  const bool known = id >= 0 && id < p.vocab;
  if (!known && threadIdx.x == 0) atomicOr(p.status, B200_STATUS_BAD_TOKEN_ID);
  const T* source = static_cast<const T*>(p.table) + (known ? id : 0) * p.width;
  const T* weight = static_cast<const T*>(p.weight);
  float* out = p.x + row * p.width;
  T* h = p.h != nullptr ? static_cast<T*>(p.h) + row * p.h_row_stride : nullptr;
  float factor = 1.0f;
  const bool quads = p.width % 4 == 0;
  if (weight != nullptr) {
    float sum = 0.0f;
    if (quads) {
      for (int c = threadIdx.x * 4; c < p.width; c += blockDim.x * 4) sum += squares_of(load_quad<T>(source + c));
    } else {
      for (int c = threadIdx.x; c < p.width; c += blockDim.x) sum += Elem<T>::load(source + c) * Elem<T>::load(source + c);
    }
    factor = 1.0f / sqrtf(block_sum(sum, scratch) / p.width + p.eps);
  }
  if (!known) factor = 0.0f;
  auto scale_at = [&](int c) { return weight != nullptr ? factor * (p.weight_offset + Elem<T>::load(weight + c)) : factor; };
  if (quads) {
    for (int c = threadIdx.x * 4; c < p.width; c += blockDim.x * 4) {
      float4 v = load_quad<T>(source + c);
      v = make_float4(v.x * scale_at(c), v.y * scale_at(c + 1), v.z * scale_at(c + 2), v.w * scale_at(c + 3));
      *reinterpret_cast<float4*>(out + c) = v;
      if (h != nullptr) store_quad<T>(h + c, v);
    }
  } else {
    for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
      const float v = Elem<T>::load(source + c) * scale_at(c);
      out[c] = v;
      if (h != nullptr) Elem<T>::store(h + c, v);
    }
  }
  if (h != nullptr)
    for (int64_t c = p.width + threadIdx.x; c < p.h_row_stride; c += blockDim.x) Elem<T>::store(h + c, 0.0f);
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

extern "C" int b200_residual_norm(void* x, const void* y, const void* y_bias, const void* post_weight,
                                  const void* next_weight, void* h, const void* summands, const int32_t* places, int64_t rows, int64_t width,
                                  int64_t splits, int64_t top, int64_t y_row_stride, int64_t h_row_stride,
                                  int64_t summand_row_stride, double epsilon, double weight_offset, int dtype,
                                  void* stream) {
  const bool adds = y != nullptr || top > 0;
  if (!x || rows < 0 || width <= 0 || splits < 0 || top < 0 || (adds && !post_weight) || (y && y_row_stride < width) ||
      (top > 0 && (!summands || !places || summand_row_stride < width)) || (h && h_row_stride < width) ||
      (next_weight && !h) || (!adds && !h))
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (width > 48 * 1024 || rows > INT32_MAX || splits > INT32_MAX || top > INT32_MAX) return B200_ERR_TOO_LARGE;
  ResidualNormParams p{static_cast<float*>(x), y, post_weight, next_weight, h, static_cast<int>(splits),
                       static_cast<int>(rows), static_cast<int>(width), y_row_stride, h_row_stride,
                       static_cast<float>(epsilon), static_cast<float>(weight_offset), summands, places,
                       static_cast<int>(top), summand_row_stride, y_bias};
  const int64_t quads = width / 4;
  if (width % 4 == 0 && quads <= 2048 && y_row_stride % 4 == 0 && h_row_stride % 4 == 0 && summand_row_stride % 4 == 0 &&
      h_row_stride - width < 32 && aligned16(x) && aligned16(y) && aligned16(h) && aligned16(post_weight) &&
      aligned16(next_weight) && aligned16(summands) && aligned16(y_bias)) {
    // few rows: a thread per four columns; many: rows of fewer, longer-working threads
    const int q = rows <= 2 * kNumSMs && quads <= 1024 ? 1 : quads <= 512 ? 2 : 4;
    const unsigned threads = static_cast<unsigned>(ceil_div(ceil_div(quads, q), 32) * 32);
    auto go = [&](auto kernel) {
      return launch_chained(kernel, dim3(static_cast<unsigned>(rows)), dim3(threads), 0,
                            static_cast<cudaStream_t>(stream), p) == cudaSuccess ? launch_status() : B200_ERR_LAUNCH;
    };
    if (dtype == B200_F32)
      return q == 1 ? go(residual_norm_quads_kernel<float, 1>) : q == 2 ? go(residual_norm_quads_kernel<float, 2>)
                                                                        : go(residual_norm_quads_kernel<float, 4>);
    return q == 1 ? go(residual_norm_quads_kernel<__nv_bfloat16, 1>)
                  : q == 2 ? go(residual_norm_quads_kernel<__nv_bfloat16, 2>) : go(residual_norm_quads_kernel<__nv_bfloat16, 4>);
  }
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
  if ((vdim == 64 || vdim == 128) && gate_row_stride % 8 == 0 && output_row_stride == heads * vdim && aligned16(input) &&
      aligned16(gate) && aligned16(output) && aligned16(weight)) {
    const dim3 blocks(static_cast<unsigned>(ceil_div(rows * heads * (vdim / 4), 256)));
    auto go = [&](auto kernel) {
      return launch_chained(kernel, blocks, dim3(256), 0, static_cast<cudaStream_t>(stream), p) == cudaSuccess
                 ? launch_status() : B200_ERR_LAUNCH;
    };
    if (dtype == B200_F32) return vdim == 64 ? go(gated_head_norm_quads_kernel<float, 64>) : go(gated_head_norm_quads_kernel<float, 128>);
    return vdim == 64 ? go(gated_head_norm_quads_kernel<__nv_bfloat16, 64>) : go(gated_head_norm_quads_kernel<__nv_bfloat16, 128>);
  }
  const dim3 grid(static_cast<unsigned>(ceil_div(rows * heads, 8)));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const cudaError_t code = dtype == B200_F32 ? launch_chained(gated_head_norm_kernel<float>, grid, dim3(256), 0, s, p)
                                             : launch_chained(gated_head_norm_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, p);
  return code == cudaSuccess ? launch_status() : B200_ERR_LAUNCH;
}

extern "C" int b200_embedding_residual(const void* table, const void* weight, const int64_t* ids, float* x, void* h,
                                       int64_t rows, int64_t width, int64_t vocab, int64_t h_row_stride,
                                       double epsilon, double weight_offset, int dtype, int32_t* status, void* stream) {
  if (!table || !ids || !x || !status || rows < 0 || width <= 0 || vocab <= 0 || (h && h_row_stride < width))
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (rows > INT32_MAX || width > INT32_MAX) return B200_ERR_TOO_LARGE;
  if (!aligned16(table) || !aligned16(x) || !aligned16(h) || h_row_stride % 4 != 0) return B200_ERR_ALIGNMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  EmbeddingParams p{table, weight, ids, x, h, static_cast<int>(width), vocab, h_row_stride, static_cast<float>(epsilon),
                    static_cast<float>(weight_offset), status};
  if (dtype == B200_F32) embedding_residual_kernel<float><<<static_cast<unsigned>(rows), 256, 0, s>>>(p);
  else embedding_residual_kernel<__nv_bfloat16><<<static_cast<unsigned>(rows), 256, 0, s>>>(p);
  return launch_status();
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
