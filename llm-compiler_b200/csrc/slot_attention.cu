// Attention over the key / value caches of a hybrid layer's slots.
//   attention_prep  bias, RMS norms over the whole query and the whole key projection, rotation of the
//                   first dimensions of every head, and the store of keys and values into the cache, in one
//                   launch behind the stacked projection (whose split-K partial sums it adds at decode
//                   sizes). Norms, angles and rotation in fp32 / fp64.
//   slot_attention  softmax attention of any rows over their slots, of any head size and dtype, on the CUDA
//                   cores: fp32 models and sizes the tensor-core kernels do not take.
// The tensor-core forms are decode_attention.cu (one row per sequence) and prefill_attention_tcgen05.cu.
#include "common.cuh"
#include "hybrid.cuh"

namespace b200 {
namespace {

struct AttentionPrepParams {
  const void* input;    // T [rows, row_stride], or fp32 [splits, rows, row_stride]
  const void* bias;     // T [row_stride] or NULL (partials only)
  const void *q_weight, *k_weight;  // T [heads * dim], [kv_heads * dim]
  const double* turns;  // [rot_dims / 2]
  void* q_out;          // T [rows, heads, size]
  void *keys, *values;  // T [slots, capacity, kv_heads, size]
  SequenceBatch batch;
  int rows, heads, kv_heads, dim, vdim, size, rot_dims, q_column, k_column, v_column, splits;
  int64_t row_stride, capacity;
  float eps;
  int32_t* status;
};

// grid (rows, 1 or 2): y = 0 the queries, y = 1 keys and values. Any sizes.
template <typename T>
__global__ void __launch_bounds__(256) attention_prep_kernel(const AttentionPrepParams p) {
  extern __shared__ float values[];  // the projection [heads * dim], then cos, sin [rot_dims / 2] each
  __shared__ float scratch[8];
  grid_launch_dependents();
  grid_dependency_wait_cta();
  const int64_t row = blockIdx.x;
  const bool is_k = blockIdx.y == 1;
  const int heads = is_k ? p.kv_heads : p.heads, count = heads * p.dim, half = p.rot_dims / 2;
  float* cosine = values + count;
  float* sine = cosine + half;
  const int sequence = p.batch.token_sequence[row];
  const int slot = p.batch.slots[sequence];
  const int64_t position = p.batch.position(sequence, row);
  auto load = [&](int column) {
    if (p.splits == 0) return Elem<T>::load(static_cast<const T*>(p.input) + row * p.row_stride + column);
    const float sum = sum_slices(static_cast<const float*>(p.input) + row * p.row_stride + column,
                                 static_cast<int64_t>(p.rows) * p.row_stride, p.splits);
    return p.bias != nullptr ? sum + Elem<T>::load(static_cast<const T*>(p.bias) + column) : sum;
  };
  T* out = static_cast<T*>(p.q_out) + row * p.heads * p.size;
  if (is_k) {
    if (slot < 0) return;
    if (position < 0 || position >= p.capacity) {
      if (threadIdx.x == 0) atomicOr(p.status, B200_STATUS_KV_OVERFLOW);
      return;
    }
    const int64_t at = (slot * p.capacity + position) * p.kv_heads * p.size;
    out = static_cast<T*>(p.keys) + at;
    T* v_out = static_cast<T*>(p.values) + at;
    for (int item = threadIdx.x; item < p.kv_heads * p.size; item += blockDim.x) {
      const int head = item / p.size, c = item - head * p.size;
      Elem<T>::store(v_out + item, c < p.vdim ? load(p.v_column + head * p.vdim + c) : 0.0f);
    }
  }
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const double turns = static_cast<double>(position) * p.turns[i];
    sincospif(2.0f * static_cast<float>(turns - rint(turns)), &sine[i], &cosine[i]);
  }
  const int column = is_k ? p.k_column : p.q_column;
  float sum = 0.0f;
  for (int item = threadIdx.x; item < count; item += blockDim.x) {
    const float v = load(column + item);
    values[item] = v;
    sum += v * v;
  }
  sum = warp_sum(sum);
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = sum;
  __syncthreads();
  sum = 0.0f;
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) sum += scratch[w];
  const float factor = 1.0f / sqrtf(sum / count + p.eps);
  const T* weight = static_cast<const T*>(is_k ? p.k_weight : p.q_weight);
  for (int item = threadIdx.x; item < heads * p.size; item += blockDim.x) {
    const int head = item / p.size, c = item - head * p.size;
    float v = 0.0f;
    if (c < p.dim) {
      const int at = head * p.dim + c;
      v = values[at] * factor * Elem<T>::load(weight + at);
      if (c < p.rot_dims) {
        const bool first = c < half;
        const int i = first ? c : c - half, other = at + (first ? half : -half);
        const float partner = values[other] * factor * Elem<T>::load(weight + other);
        v = v * cosine[i] + (first ? -partner : partner) * sine[i];
      }
    }
    Elem<T>::store(out + item, v);
  }
}

// The same for sizes in whole quads: a CTA per row holds the projection in registers, Q quads a thread (the
// queries' first, then the keys', then the values'), every load in flight at once.
template <typename T>
struct RawQuad { using type = float4; };
template <>
struct RawQuad<__nv_bfloat16> { using type = uint2; };
__device__ __forceinline__ float4 widen(float4 v) { return v; }
__device__ __forceinline__ float4 widen(uint2 t) { return make_float4(bf16_lo(t.x), bf16_hi(t.x), bf16_lo(t.y), bf16_hi(t.y)); }
template <typename T>
__device__ __forceinline__ float4 read_quad(const T* p) {
  return widen(*reinterpret_cast<const typename RawQuad<T>::type*>(p));
}
template <typename T>
__device__ __forceinline__ void write_quad(T* p, float4 v) {
  if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(p) = v;
  else *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// PLAIN: dim, vdim and the row size are one power of two.
template <typename T, int Q, bool PLAIN>
__global__ void __launch_bounds__(512) attention_prep_quads_kernel(const AttentionPrepParams p) {
  extern __shared__ __align__(16) float normed[];  // q and k [(heads + kv_heads) * dim], then cos, sin [rot_dims / 2] each
  __shared__ float scratch[2][16], factors[2];
  const int dq = p.dim / 4, half = p.rot_dims / 2;
  const bool kv = p.keys != nullptr;
  const int nq = p.heads * dq, nk = kv ? p.kv_heads * dq : 0, nv = kv ? p.kv_heads * (p.vdim / 4) : 0;
  float* cosine = normed + (nq + nk) * 4;
  float* sine = cosine + half;
  grid_launch_dependents();
  grid_dependency_wait_cta();
  const int64_t row = blockIdx.x;
  const int sequence = p.batch.token_sequence[row];
  auto column_of = [&](int i) {
    return i < nq ? p.q_column + i * 4 : i < nq + nk ? p.k_column + (i - nq) * 4 : p.v_column + (i - nq - nk) * 4;
  };
  float4 v[Q];
#pragma unroll
  for (int j = 0; j < Q; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    v[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (i >= nq + nk + nv) continue;
    const int column = column_of(i);
    if (p.splits > 0) {
      const float* in = static_cast<const float*>(p.input) + row * p.row_stride + column;
      const int64_t slice = static_cast<int64_t>(p.rows) * p.row_stride;
      if (p.bias != nullptr) v[j] = read_quad<T>(static_cast<const T*>(p.bias) + column);
      for (int s = 0; s < p.splits; s += 4) {
        float4 t[4];
#pragma unroll
        for (int e = 0; e < 4; ++e)
          t[e] = s + e < p.splits ? __ldcg(reinterpret_cast<const float4*>(in + (s + e) * slice))
                                  : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          v[j].x += t[e].x; v[j].y += t[e].y; v[j].z += t[e].z; v[j].w += t[e].w;
        }
      }
    } else {
      v[j] = read_quad<T>(static_cast<const T*>(p.input) + row * p.row_stride + column);
    }
  }
  using Raw = typename RawQuad<T>::type;
  const Raw* q_weight = static_cast<const Raw*>(p.q_weight);
  const Raw* k_weight = static_cast<const Raw*>(p.k_weight);
  Raw weight[Q];
#pragma unroll
  for (int j = 0; j < Q; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < nq + nk) weight[j] = i < nq ? q_weight[i] : k_weight[i - nq];
  }
  const int slot = p.batch.slots[sequence];
  const int64_t position = p.batch.position(sequence, row);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const double turns = static_cast<double>(position) * p.turns[i];
    sincospif(2.0f * static_cast<float>(turns - rint(turns)), &sine[i], &cosine[i]);
  }
  float q_sum = 0.0f, k_sum = 0.0f;
#pragma unroll
  for (int j = 0; j < Q; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    const float squares = v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    if (i < nq) q_sum += squares;
    else if (i < nq + nk) k_sum += squares;
  }
  q_sum = warp_sum(q_sum);
  k_sum = warp_sum(k_sum);
  const int warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  if ((threadIdx.x & 31) == 0) {
    scratch[0][warp] = q_sum;
    scratch[1][warp] = k_sum;
  }
  __syncthreads();
  if (warp == 0) {  // half a warp for each of the two
    const int lane = threadIdx.x & 31, which = lane >> 4;
    float sum = (lane & 15) < warps ? scratch[which][lane & 15] : 0.0f;
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if ((lane & 15) == 0) factors[which] = 1.0f / sqrtf(sum / ((which == 0 ? p.heads : p.kv_heads) * p.dim) + p.eps);
  }
  __syncthreads();
#pragma unroll
  for (int j = 0; j < Q; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i >= nq + nk) continue;
    const float4 w = widen(weight[j]);
    const float f = factors[i < nq ? 0 : 1];
    v[j] = make_float4(v[j].x * f * w.x, v[j].y * f * w.y, v[j].z * f * w.z, v[j].w * f * w.w);
    *reinterpret_cast<float4*>(normed + i * 4) = v[j];
  }
  __syncthreads();
  const bool inside = slot >= 0 && position >= 0 && position < p.capacity;
  if (kv && slot >= 0 && !inside && threadIdx.x == 0) atomicOr(p.status, B200_STATUS_KV_OVERFLOW);
  const int64_t cache = (slot * p.capacity + position) * p.kv_heads * p.size;
  T* q_out = static_cast<T*>(p.q_out) + row * p.heads * p.size;
  T* k_out = static_cast<T*>(p.keys) + cache;
  T* v_out = static_cast<T*>(p.values) + cache;
#pragma unroll
  for (int j = 0; j < Q; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i >= nq + nk + nv || (i >= nq && !inside)) continue;
    if (i >= nq + nk) {
      const int quad = i - nq - nk, head = PLAIN ? 0 : quad / (p.vdim / 4);
      write_quad<T>(v_out + head * p.size + (quad - head * (p.vdim / 4)) * 4, v[j]);
      continue;
    }
    const int quad = i < nq ? i : i - nq;
    const int head = PLAIN ? 0 : quad / dq, within = quad - head * dq;  // (PLAIN: heads lie side by side)
    const int c = (PLAIN ? quad & (dq - 1) : within) * 4;
    float4 out = v[j];
    if (c < p.rot_dims) {
      const bool first = c < half;
      const int at = first ? c : c - half;
      const float4 other = *reinterpret_cast<const float4*>(normed + i * 4 + (first ? half : -half));
      const float4 cs = *reinterpret_cast<const float4*>(cosine + at);
      float4 sn = *reinterpret_cast<const float4*>(sine + at);
      if (first) sn = make_float4(-sn.x, -sn.y, -sn.z, -sn.w);
      out = make_float4(out.x * cs.x + other.x * sn.x, out.y * cs.y + other.y * sn.y, out.z * cs.z + other.z * sn.z,
                        out.w * cs.w + other.w * sn.w);
    }
    write_quad<T>((i < nq ? q_out : k_out) + head * p.size + within * 4, out);
  }
  if (PLAIN) return;
  // zeros behind every head's dim / vdim
  if (p.size > p.dim) {
    const int pad = (p.size - p.dim) / 4;
    for (int i = threadIdx.x; i < p.heads * pad; i += blockDim.x)
      write_quad<T>(q_out + i / pad * p.size + p.dim + i % pad * 4, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
    for (int i = threadIdx.x; kv && inside && i < p.kv_heads * pad; i += blockDim.x)
      write_quad<T>(k_out + i / pad * p.size + p.dim + i % pad * 4, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
  }
  if (kv && inside && p.size > p.vdim) {
    const int pad = (p.size - p.vdim) / 4;
    for (int i = threadIdx.x; i < p.kv_heads * pad; i += blockDim.x)
      write_quad<T>(v_out + i / pad * p.size + p.vdim + i % pad * 4, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
  }
}

// ---- CUDA-core attention -----------------------------------------------------------------
constexpr int kSlotWarps = 4, kSlotValues = 16;  // value columns a lane holds: head sizes up to 512

template <typename T>
__global__ void __launch_bounds__(kSlotWarps * 32)
slot_attention_kernel(const T* q, const T* keys, const T* values, T* out, SequenceBatch batch, int heads, int kv_heads,
                      int size, int64_t capacity, int chunk, float scale) {
  extern __shared__ float shared[];  // query [size], then per warp: output [size], maximum, sum
  const int64_t row = blockIdx.x;
  const int head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int sequence = batch.token_sequence[row];
  const int slot = batch.slots[sequence];
  T* to = out + (row * heads + head) * size;
  if (slot < 0) {
    for (int c = threadIdx.x; c < size; c += blockDim.x) Elem<T>::store(to + c, 0.0f);
    return;
  }
  int64_t position = batch.position(sequence, row);
  if (position >= capacity) position = capacity - 1;
  const int64_t first = chunk > 0 ? position / chunk * chunk : 0;
  const int64_t token = static_cast<int64_t>(kv_heads) * size;
  const int64_t base = slot * capacity * token + (head / (heads / kv_heads)) * size;
  float* query = shared;
  for (int c = threadIdx.x; c < size; c += blockDim.x) query[c] = Elem<T>::load(q + (row * heads + head) * size + c) * scale;
  __syncthreads();
  float maximum = -INFINITY, sum = 0.0f, acc[kSlotValues];
#pragma unroll
  for (int i = 0; i < kSlotValues; ++i) acc[i] = 0.0f;
  for (int64_t j = first + warp; j <= position; j += kSlotWarps) {
    const T* key = keys + base + j * token;
    const T* value = values + base + j * token;
    float score = 0.0f;
    for (int c = lane; c < size; c += 32) score = fmaf(query[c], Elem<T>::load(key + c), score);
    score = warp_sum(score);
    const float top = fmaxf(maximum, score);
    const float keep = expf(maximum - top), weight = expf(score - top);  // (expf(-inf) = 0)
    maximum = top;
    sum = sum * keep + weight;
#pragma unroll
    for (int i = 0; i < kSlotValues; ++i) {
      const int c = lane + 32 * i;
      if (c < size) acc[i] = fmaf(weight, Elem<T>::load(value + c), acc[i] * keep);
    }
  }
  float* own = shared + size + warp * (size + 2);
#pragma unroll
  for (int i = 0; i < kSlotValues; ++i)
    if (lane + 32 * i < size) own[lane + 32 * i] = acc[i];
  if (lane == 0) {
    own[size] = maximum;
    own[size + 1] = sum;
  }
  __syncthreads();
  float top = -INFINITY, total = 0.0f;
  for (int w = 0; w < kSlotWarps; ++w) top = fmaxf(top, shared[size + w * (size + 2) + size]);
  for (int w = 0; w < kSlotWarps; ++w) {
    const float* part = shared + size + w * (size + 2);
    total += part[size + 1] * expf(part[size] - top);
  }
  for (int c = threadIdx.x; c < size; c += blockDim.x) {
    float v = 0.0f;
    for (int w = 0; w < kSlotWarps; ++w) {
      const float* part = shared + size + w * (size + 2);
      v += part[c] * expf(part[size] - top);
    }
    Elem<T>::store(to + c, v / total);
  }
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int b200_attention_prep(const b200_attention_prep_inputs* in, int dtype, int32_t* status, void* stream) {
  if (in == nullptr || !in->input || !in->q_weight || !in->q_out || !in->token_sequence || !in->starts || !in->slots ||
      !in->bases || !status || in->rows < 0 || in->heads <= 0 || in->kv_heads <= 0 || in->heads % in->kv_heads != 0 ||
      in->dim <= 0 || in->row_size < in->dim || in->rot_dims < 0 || in->rot_dims > in->dim || in->rot_dims % 2 != 0 ||
      (in->rot_dims > 0 && !in->turns) || in->splits < 0 || in->q_column < 0 ||
      in->row_stride < in->q_column + in->heads * in->dim)
    return B200_ERR_BAD_ARGUMENT;
  const bool kv = in->keys != nullptr;
  if (kv && (!in->values || !in->k_weight || in->vdim <= 0 || in->row_size < in->vdim || in->capacity <= 0 ||
             in->k_column < 0 || in->v_column < 0 || in->row_stride < in->k_column + in->kv_heads * in->dim ||
             in->row_stride < in->v_column + in->kv_heads * in->vdim))
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (in->rows == 0) return B200_OK;
  if (in->rows > INT32_MAX || in->heads * in->row_size > INT32_MAX) return B200_ERR_TOO_LARGE;
  const int64_t smem = (in->heads * in->dim + in->rot_dims) * static_cast<int64_t>(sizeof(float));
  if (smem > 200 * 1024) return B200_ERR_TOO_LARGE;
  AttentionPrepParams p{in->input, in->bias, in->q_weight, in->k_weight, in->turns, in->q_out, in->keys, in->values,
                        {in->token_sequence, in->starts, in->slots, in->bases}, static_cast<int>(in->rows),
                        static_cast<int>(in->heads), static_cast<int>(in->kv_heads), static_cast<int>(in->dim),
                        static_cast<int>(in->vdim), static_cast<int>(in->row_size), static_cast<int>(in->rot_dims),
                        static_cast<int>(in->q_column), static_cast<int>(in->k_column), static_cast<int>(in->v_column),
                        static_cast<int>(in->splits), in->row_stride, in->capacity, static_cast<float>(in->epsilon), status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool whole = in->dim % 4 == 0 && (!kv || in->vdim % 4 == 0) && in->row_size % 4 == 0 && in->q_column % 4 == 0 &&
                     in->k_column % 4 == 0 && in->v_column % 4 == 0 && in->row_stride % 4 == 0 && aligned16(in->input) &&
                     aligned16(in->bias) && aligned16(in->q_weight) && aligned16(in->k_weight) && aligned16(in->q_out) &&
                     aligned16(in->keys) && aligned16(in->values);
  const int64_t quads = (in->heads * in->dim + (kv ? in->kv_heads * (in->dim + in->vdim) : 0)) / 4;
  const int64_t quads_smem = (in->heads * in->dim + (kv ? in->kv_heads * in->dim : 0) + in->rot_dims) * static_cast<int64_t>(sizeof(float));
  if (whole && in->rot_dims % 8 == 0 && quads <= 4096 && quads_smem <= 200 * 1024) {
    const bool plain = (in->dim & (in->dim - 1)) == 0 && in->row_size == in->dim && (!kv || in->vdim == in->dim);
    // few rows: a thread per quad or two; many: CTAs of a few warps, four quads a thread
    const int64_t q = quads > 2048 ? 8 : in->rows <= 2 * kNumSMs && quads <= 1024 ? 2 : 4;
    const int64_t threads = ceil_div(ceil_div(quads, q), 32) * 32;
    auto go = [&](auto kernel) {
      if (quads_smem > 48 * 1024 &&
          cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(quads_smem)) != cudaSuccess)
        return B200_ERR_LAUNCH;
      return launch_chained(kernel, dim3(static_cast<unsigned>(in->rows)), dim3(static_cast<unsigned>(threads)),
                            static_cast<size_t>(quads_smem), s, p) == cudaSuccess ? launch_status() : B200_ERR_LAUNCH;
    };
    auto pick = [&](auto tag) {
      using T = typename decltype(tag)::type;
      if (plain) return q == 2 ? go(attention_prep_quads_kernel<T, 2, true>) : q == 4 ? go(attention_prep_quads_kernel<T, 4, true>)
                                                                                      : go(attention_prep_quads_kernel<T, 8, true>);
      return q == 2 ? go(attention_prep_quads_kernel<T, 2, false>) : q == 4 ? go(attention_prep_quads_kernel<T, 4, false>)
                                                                            : go(attention_prep_quads_kernel<T, 8, false>);
    };
    return dtype == B200_F32 ? pick(TypeTag<float>{}) : pick(TypeTag<__nv_bfloat16>{});
  }
  const dim3 grid(static_cast<unsigned>(in->rows), kv ? 2u : 1u);
  auto go = [&](auto kernel) {
    if (smem > 48 * 1024 &&
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)
      return B200_ERR_LAUNCH;
    return launch_chained(kernel, grid, dim3(256), static_cast<size_t>(smem), s, p) == cudaSuccess ? launch_status()
                                                                                                    : B200_ERR_LAUNCH;
  };
  return dtype == B200_F32 ? go(attention_prep_kernel<float>) : go(attention_prep_kernel<__nv_bfloat16>);
}

extern "C" int b200_slot_attention(const void* q, const void* keys, const void* values, void* out,
                                   const int32_t* token_sequence, const int32_t* starts, const int32_t* slots,
                                   const int32_t* bases, int64_t rows, int64_t heads, int64_t kv_heads, int64_t row_size,
                                   int64_t capacity, int64_t chunk, double scale, int dtype, void* stream) {
  if (!q || !keys || !values || !out || !token_sequence || !starts || !slots || !bases || rows < 0 || heads <= 0 ||
      kv_heads <= 0 || heads % kv_heads != 0 || row_size <= 0 || capacity <= 0 || chunk < 0)
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (row_size > 32 * kSlotValues || heads > 65535 || rows > INT32_MAX || chunk > INT32_MAX) return B200_ERR_TOO_LARGE;
  if (rows == 0) return B200_OK;
  const dim3 grid(static_cast<unsigned>(rows), static_cast<unsigned>(heads));
  const size_t smem = (row_size + kSlotWarps * (row_size + 2)) * sizeof(float);
  const SequenceBatch batch{token_sequence, starts, slots, bases};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto go = [&](auto tag) {
    using T = typename decltype(tag)::type;
    slot_attention_kernel<T><<<grid, kSlotWarps * 32, smem, s>>>(
        static_cast<const T*>(q), static_cast<const T*>(keys), static_cast<const T*>(values), static_cast<T*>(out), batch,
        static_cast<int>(heads), static_cast<int>(kv_heads), static_cast<int>(row_size), capacity, static_cast<int>(chunk),
        static_cast<float>(scale));
    return launch_status();
  };
  return dtype == B200_F32 ? go(TypeTag<float>{}) : go(TypeTag<__nv_bfloat16>{});
}
