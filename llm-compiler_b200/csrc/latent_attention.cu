// Latent attention over the cached latents (one row of kv_rank values per token, shared by all heads),
// in the absorbed form: a head's query is carried into the latent space (q W_uk), scored against the
// cached rows themselves, and the weighted sum of the rows is carried out of it (W_uv) behind the
// attention. The softmax denominator may hold a learned term per head (a sink) beside the keys.
//
// This file: the per-head projections in and out of the latent space, and attention for any rank up to
// 1024 on the CUDA cores (fp32 models, and shapes the tensor-core kernel does not take).
#include "common.cuh"
#include "hybrid.cuh"

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
  if (dtype == B200_F32) head_linear_kernel<float><<<grid, 256, 0, s>>>(p);
  else head_linear_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(p);
  return launch_status();
}

extern "C" int b200_latent_attention(const void* q, const void* cache, const void* sink, void* out,
                                     const int32_t* token_sequence, const int32_t* starts, const int32_t* slots,
                                     const int32_t* bases, int64_t rows, int64_t heads, int64_t rank_row,
                                     int64_t capacity, double scale, int dtype, void* stream) {
  if (!q || !cache || !out || !token_sequence || !starts || !slots || !bases || rows < 0 || heads <= 0 ||
      rank_row <= 0 || capacity <= 0)
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (rows > INT32_MAX || heads > 65535) return B200_ERR_TOO_LARGE;
  LatentAttentionParams p{q, cache, sink, out, {token_sequence, starts, slots, bases}, static_cast<int>(heads),
                          static_cast<int>(rank_row), capacity, static_cast<float>(scale)};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == B200_F32 ? launch_generic<float>(p, rows, s) : launch_generic<__nv_bfloat16>(p, rows, s);
}
