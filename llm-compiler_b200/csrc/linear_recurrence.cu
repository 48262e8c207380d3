// Linear recurrences with a matrix state per head, S [dim, vdim] in fp32:
//   retention      S' = gamma_h S + k v^T,                                      read-out S'^T q
//   gated delta    P = diag(g) S, S' = P + k (beta (v - P^T k))^T,             read-out S'^T q
//                  (g: a decay per key channel, or one for all channels of a head)
// The columns of S are independent of each other, so a CTA owns a slice of them and walks the tokens.
//
// This file: the operand preparation (rotation, short convolution, unit norm, decays) and the token by
// token scan, exact fp32 throughout, for any dim up to 512; it serves fp32 models and short portions.
#include "common.cuh"
#include "hybrid.cuh"
#include "recurrence.cuh"

namespace b200 {
namespace {

// ---- operand preparation ------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) retention_prep_kernel(const RetentionInputs p, float* q,
                                                             float* k, float* v) {
  extern __shared__ float rotation[];  // cos, sin of this row's position [rot_dims / 2] each
  const int64_t row = blockIdx.x;
  const int half = p.rot_dims / 2;
  const int64_t position = p.batch.position(p.batch.token_sequence[row], row);
  for (int i = threadIdx.x; i < half; i += blockDim.x)
    rotation_of(position, i, p.rot_dims, p.log2_base, rotation[i], rotation[half + i]);
  __syncthreads();
  const T* in = static_cast<const T*>(p.input) + row * p.row_stride;
  const int qk = p.heads * p.dim;
  for (int c = threadIdx.x; c < 2 * qk; c += blockDim.x) {
    const bool is_k = c >= qk;
    const int channel = is_k ? c - qk : c;
    const int within = channel % p.dim;
    const T* src = in + (is_k ? p.k_column : p.q_column) + channel;
    float value = Elem<T>::load(src);
    if (within < half)
      value = value * rotation[within] - Elem<T>::load(src + half) * rotation[half + within];
    else if (within < p.rot_dims)
      value = value * rotation[within - half] + Elem<T>::load(src - half) * rotation[within];
    if (is_k) k[row * qk + channel] = value * p.k_scale;
    else q[row * qk + channel] = value;
  }
  for (int c = threadIdx.x; c < p.heads * p.vdim; c += blockDim.x)
    v[row * p.heads * p.vdim + c] = Elem<T>::load(in + p.v_column + c);
}

// One warp per unit of a row: a q head, a k head, a v head, or a head's step size and decays.
template <typename T>
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaInputs p, float* q, float* k, float* v,
                                                         float* beta, float* log_decay) {
  const int64_t row = blockIdx.x;
  const int lane = threadIdx.x & 31;
  const int sequence = p.batch.token_sequence[row];
  const int slot = p.batch.slots[sequence];
  const int64_t position = p.batch.position(sequence, row);
  const int64_t local = row - p.batch.starts[sequence];
  const int units = 2 * p.kv_heads + 2 * p.heads;
  for (int unit = threadIdx.x >> 5; unit < units; unit += blockDim.x >> 5) {
    if (unit < 2 * p.kv_heads) {
      const bool is_k = unit >= p.kv_heads;
      const int head = is_k ? unit - p.kv_heads : unit;
      float* out = (is_k ? k : q) + (row * p.kv_heads + head) * p.dim;
      float sum = 0.0f;
      for (int c = lane; c < p.dim; c += 32) {
        const float value = slot < 0 ? 0.0f : silu_of(short_conv<T>(p, is_k ? 1 : 0, head * p.dim + c, row, local, position, slot));
        out[c] = value;
        sum += value * value;
      }
      float factor = 1.0f / sqrtf(warp_sum(sum) + kUnitEpsilon);
      if (!is_k) factor *= p.q_scale;
      for (int c = lane; c < p.dim; c += 32) out[c] *= factor;
    } else if (unit < 2 * p.kv_heads + p.heads) {
      const int head = unit - 2 * p.kv_heads;
      for (int c = lane; c < p.vdim; c += 32)
        v[(row * p.heads + head) * p.vdim + c] =
            slot < 0 ? 0.0f : silu_of(short_conv<T>(p, 2, head * p.vdim + c, row, local, position, slot));
    } else {
      const int head = unit - 2 * p.kv_heads - p.heads;
      if (lane == 0) beta[row * p.heads + head] = delta_beta<T>(p, row, head);
      for (int c = lane; c < p.decay_dim; c += 32)
        log_decay[(row * p.heads + head) * p.decay_dim + c] = delta_log_decay<T>(p, row, head, c);
    }
  }
}

// bf16 prompts with dim = vdim = 32 CPL and at most four taps: a warp walks 32 tokens of one unit (a q,
// k or v head, or a head's decays) with the convolution's window in registers, CPL channels a lane, eight
// tokens' loads in flight.
template <int CPL>
__device__ __forceinline__ void load_channels(const __nv_bfloat16* p, float (&v)[CPL]) {
  if (CPL == 4) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    v[0] = bf16_lo(t.x); v[1] = bf16_hi(t.x); v[CPL - 2] = bf16_lo(t.y); v[CPL - 1] = bf16_hi(t.y);
  } else {
    const uint32_t t = *reinterpret_cast<const uint32_t*>(p);
    v[0] = bf16_lo(t); v[1] = bf16_hi(t);
  }
}
template <int CPL>
__device__ __forceinline__ void store_channels(float* p, const float (&v)[CPL]) {
  if (CPL == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[CPL - 2], v[CPL - 1]);
  else *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
}

template <int CPL>
__global__ void __launch_bounds__(256) delta_prep_tiled_kernel(const DeltaInputs p, float* q, float* k, float* v,
                                                               float* beta, float* log_decay) {
  constexpr int kDim = 32 * CPL, kTokens = 32, kBatch = 8, kTaps = 4;
  const int lane = threadIdx.x & 31, sequence = blockIdx.z;
  const int unit = blockIdx.y * 8 + (threadIdx.x >> 5);
  const int slot = p.batch.slots[sequence];
  const int64_t first = p.batch.starts[sequence], last = p.batch.starts[sequence + 1];
  const int64_t row0 = first + static_cast<int64_t>(blockIdx.x) * kTokens;
  if (unit >= 2 * p.kv_heads + 2 * p.heads || row0 >= last || slot < 0) return;
  const int count = last - row0 < kTokens ? static_cast<int>(last - row0) : kTokens;
  const int c = lane * CPL;
  if (unit >= 2 * p.kv_heads + p.heads) {  // step size and decays
    const int head = unit - 2 * p.kv_heads - p.heads;
    if (lane < count) beta[(row0 + lane) * p.heads + head] = delta_beta<__nv_bfloat16>(p, row0 + lane, head);
    if (p.decay_dim == 1) {
      if (lane < count) log_decay[(row0 + lane) * p.heads + head] = delta_log_decay<__nv_bfloat16>(p, row0 + lane, head, 0);
      return;
    }
    const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(p.gates) + p.decay_column + head * kDim + c;
    float bias[CPL];
    load_channels<CPL>(static_cast<const __nv_bfloat16*>(p.dt_bias) + head * kDim + c, bias);
    const float rate = -expf(__bfloat162float(static_cast<const __nv_bfloat16*>(p.a_log)[head]));
    for (int t0 = 0; t0 < count; t0 += kBatch) {
      float step[kBatch][CPL];
#pragma unroll
      for (int t = 0; t < kBatch; ++t)
        if (t0 + t < count) load_channels<CPL>(in + (row0 + t0 + t) * p.gate_row_stride, step[t]);
#pragma unroll
      for (int t = 0; t < kBatch; ++t) {
        if (t0 + t >= count) break;
#pragma unroll
        for (int i = 0; i < CPL; ++i) step[t][i] = rate * softplus_f32(step[t][i] + bias[i]);
        store_channels<CPL>(log_decay + ((row0 + t0 + t) * p.heads + head) * kDim + c, step[t]);
      }
    }
    return;
  }
  const int which = unit < p.kv_heads ? 0 : unit < 2 * p.kv_heads ? 1 : 2;
  const int head = unit - which * p.kv_heads;
  const int channel = head * kDim + c;
  const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(p.input) +
                            (which == 0 ? p.q_column : which == 1 ? p.k_column : p.v_column) + channel;
  const __nv_bfloat16* taps = static_cast<const __nv_bfloat16*>(which == 0 ? p.q_conv : which == 1 ? p.k_conv : p.v_conv);
  float weight[CPL][kTaps], window[kTaps - 1][CPL];  // weight[.][b]: of the input b tokens back; window: 1, 2, 3 back
#pragma unroll
  for (int i = 0; i < CPL; ++i)
#pragma unroll
    for (int b = 0; b < kTaps; ++b)
      weight[i][b] = b < p.taps ? __bfloat162float(taps[(channel + i) * p.taps + p.taps - 1 - b]) : 0.0f;
  const int64_t position = p.batch.position(sequence, row0);
  const int qk = p.kv_heads * p.dim, channels = 2 * qk + p.heads * p.vdim;
  const __nv_bfloat16* ring = static_cast<const __nv_bfloat16*>(p.ring) + static_cast<int64_t>(slot) * p.taps * channels + which * qk + channel;
#pragma unroll
  for (int b = 1; b < kTaps; ++b) {
#pragma unroll
    for (int i = 0; i < CPL; ++i) window[b - 1][i] = 0.0f;
    if (b >= p.taps || b > position) continue;
    if (row0 - b >= first) load_channels<CPL>(in + (row0 - b) * p.row_stride, window[b - 1]);
    else load_channels<CPL>(ring + static_cast<int>((position - b) % p.taps) * static_cast<int64_t>(channels), window[b - 1]);
  }
  float* out = which == 0 ? q : which == 1 ? k : v;
  const int out_heads = which == 2 ? p.heads : p.kv_heads;
  for (int t0 = 0; t0 < count; t0 += kBatch) {
    float raw[kBatch][CPL];
#pragma unroll
    for (int t = 0; t < kBatch; ++t)
      if (t0 + t < count) load_channels<CPL>(in + (row0 + t0 + t) * p.row_stride, raw[t]);
#pragma unroll
    for (int t = 0; t < kBatch; ++t) {
      if (t0 + t >= count) break;
      float y[CPL], sum = 0.0f;
#pragma unroll
      for (int i = 0; i < CPL; ++i) {
        y[i] = silu_of(weight[i][0] * raw[t][i] + weight[i][1] * window[0][i] + weight[i][2] * window[1][i] + weight[i][3] * window[2][i]);
        sum += y[i] * y[i];
        window[2][i] = window[1][i];
        window[1][i] = window[0][i];
        window[0][i] = raw[t][i];
      }
      if (which < 2) {
        float factor = 1.0f / sqrtf(warp_sum(sum) + kUnitEpsilon);
        if (which == 0) factor *= p.q_scale;
#pragma unroll
        for (int i = 0; i < CPL; ++i) y[i] *= factor;
      }
      store_channels<CPL>(out + ((row0 + t0 + t) * out_heads + head) * kDim + c, y);
    }
  }
}

// The last taps inputs of every sequence into its ring (entry position % taps), behind the kernels
// that still read the ring's older entries.
template <typename T>
__global__ void __launch_bounds__(256) conv_tail_kernel(const DeltaInputs p) {
  const int sequence = blockIdx.x;
  const int slot = p.batch.slots[sequence];
  if (slot < 0) return;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  const int64_t first = p.batch.starts[sequence], last = p.batch.starts[sequence + 1];
  const int64_t begin = last - first > p.taps ? last - p.taps : first;
  const int channels = 2 * p.kv_heads * p.dim + p.heads * p.vdim;
  for (int64_t row = begin; row < last; ++row) {
    const int64_t entry = p.batch.position(sequence, row) % p.taps;
    T* ring = static_cast<T*>(p.ring) + (slot * p.taps + entry) * channels;
    const T* in = static_cast<const T*>(p.input) + row * p.row_stride;
    if (c < channels) {
      const int qk = p.kv_heads * p.dim;
      const int column = c < qk ? p.q_column + c : (c < 2 * qk ? p.k_column + c - qk : p.v_column + c - 2 * qk);
      ring[c] = in[column];
    }
  }
}

// ---- token by token scan ----------------------------------------------------------------
constexpr int kScanThreads = 128, kScanColumns = 8, kScanTokens = 16;

struct ScanParams {
  const float *q, *k, *v;     // [rows, kv_heads, dim] x 2, [rows, heads, vdim]
  const float* beta;          // [rows, heads]            (delta)
  const float* log_decay;     // [rows, heads, decay_dim] natural log (delta); [heads] decay itself (retention)
  float* state;               // [slots, heads, dim, state_row]
  float* output;              // [rows, heads, vdim]
  SequenceBatch batch;
  int heads, kv_heads, dim, vdim, state_row, decay_dim;
};

// 16 lanes share a column: lane g holds rows g, g + 16, ... A column's sums are four shuffles.
template <int R, bool DELTA>
__global__ void __launch_bounds__(kScanThreads) recurrence_scan_kernel(const ScanParams p) {
  extern __shared__ float tile[];  // per token: k [dim], q [dim], decay [dim] (delta), v [columns], beta
  const int head = blockIdx.y, sequence = blockIdx.z;
  const int group = threadIdx.x & 15, column = blockIdx.x * kScanColumns + (threadIdx.x >> 4);
  const int kv_head = head / (p.heads / p.kv_heads);
  const int slot = p.batch.slots[sequence];
  const int64_t first = p.batch.starts[sequence], last = p.batch.starts[sequence + 1];
  const bool own = column < p.vdim;
  if (slot < 0) {
    for (int64_t row = first; row < last; ++row)
      if (own && group == 0) p.output[(row * p.heads + head) * p.vdim + column] = 0.0f;
    return;
  }
  const int stride = (DELTA ? 3 : 2) * p.dim + kScanColumns + 1;
  float* state = p.state + (static_cast<int64_t>(slot) * p.heads + head) * p.dim * p.state_row + column;
  float s[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = group + 16 * i;
    s[i] = own && r < p.dim && p.batch.bases[sequence] > 0 ? state[static_cast<int64_t>(r) * p.state_row] : 0.0f;
  }
  const float head_decay = DELTA ? 0.0f : p.log_decay[head];
  for (int64_t row0 = first; row0 < last; row0 += kScanTokens) {
    const int count = static_cast<int>(last - row0 < kScanTokens ? last - row0 : kScanTokens);
    __syncthreads();
    for (int item = threadIdx.x; item < count * p.dim; item += kScanThreads) {
      const int t = item / p.dim, c = item % p.dim;
      const int64_t source = ((row0 + t) * p.kv_heads + kv_head) * p.dim + c;
      tile[t * stride + c] = p.k[source];
      tile[t * stride + p.dim + c] = p.q[source];
      if (DELTA) tile[t * stride + 2 * p.dim + c] = expf(p.log_decay[((row0 + t) * p.heads + head) * p.decay_dim + (p.decay_dim == 1 ? 0 : c)]);
    }
    for (int item = threadIdx.x; item < count * (kScanColumns + 1); item += kScanThreads) {
      const int t = item / (kScanColumns + 1), c = item % (kScanColumns + 1);
      const int64_t unit = (row0 + t) * p.heads + head;
      float value = 0.0f;
      if (c == kScanColumns) {
        if (DELTA) value = p.beta[unit];
      } else if (blockIdx.x * kScanColumns + c < p.vdim) {
        value = p.v[unit * p.vdim + blockIdx.x * kScanColumns + c];
      }
      tile[t * stride + (DELTA ? 3 : 2) * p.dim + c] = value;
    }
    __syncthreads();
    for (int t = 0; t < count; ++t) {
      const float* k = tile + t * stride;
      const float* q = k + p.dim;
      const float* rest = k + (DELTA ? 3 : 2) * p.dim;
      float u = rest[threadIdx.x >> 4];
      if (DELTA) {
        const float* g = q + p.dim;
        float along = 0.0f;
#pragma unroll
        for (int i = 0; i < R; ++i) {
          const int r = group + 16 * i;
          if (r < p.dim) {
            s[i] *= g[r];
            along = fmaf(s[i], k[r], along);
          }
        }
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) along += __shfl_xor_sync(0xffffffffu, along, o);
        u = rest[kScanColumns] * (u - along);
      }
      float out = 0.0f;
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int r = group + 16 * i;
        if (r < p.dim) {
          s[i] = DELTA ? fmaf(k[r], u, s[i]) : fmaf(k[r], u, head_decay * s[i]);
          out = fmaf(s[i], q[r], out);
        }
      }
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) out += __shfl_xor_sync(0xffffffffu, out, o);
      if (own && group == 0) p.output[((row0 + t) * p.heads + head) * p.vdim + column] = out;
    }
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = group + 16 * i;
    if (own && r < p.dim) state[static_cast<int64_t>(r) * p.state_row] = s[i];
  }
}

template <int R, bool DELTA>
int launch_scan(const ScanParams& p, int64_t sequences, cudaStream_t stream) {
  const int smem = kScanTokens * ((DELTA ? 3 : 2) * p.dim + kScanColumns + 1) * static_cast<int>(sizeof(float));
  auto kernel = recurrence_scan_kernel<R, DELTA>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
    return B200_ERR_LAUNCH;
  const dim3 grid(static_cast<unsigned>(ceil_div(p.vdim, kScanColumns)), static_cast<unsigned>(p.heads),
                  static_cast<unsigned>(sequences));
  kernel<<<grid, kScanThreads, smem, stream>>>(p);
  return launch_status();
}

template <bool DELTA>
int dispatch_scan(const ScanParams& p, int64_t sequences, cudaStream_t stream) {
  if (p.dim <= 64) return launch_scan<4, DELTA>(p, sequences, stream);
  if (p.dim <= 128) return launch_scan<8, DELTA>(p, sequences, stream);
  if (p.dim <= 256) return launch_scan<16, DELTA>(p, sequences, stream);
  if (p.dim <= 512) return launch_scan<32, DELTA>(p, sequences, stream);
  return B200_ERR_TOO_LARGE;
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int b200_retention_prep(const b200_retention_inputs* inputs, float* q, float* k, float* v,
                                   int64_t rows, int dtype, void* stream) {
  RetentionInputs p;
  if (!retention_inputs_from(inputs, &p) || !q || !k || !v || rows < 0) return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (rows > INT32_MAX) return B200_ERR_TOO_LARGE;
  const size_t smem = (p.rot_dims + 1) * sizeof(float);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_F32) retention_prep_kernel<float><<<static_cast<unsigned>(rows), 256, smem, s>>>(p, q, k, v);
  else retention_prep_kernel<__nv_bfloat16><<<static_cast<unsigned>(rows), 256, smem, s>>>(p, q, k, v);
  return launch_status();
}

extern "C" int b200_delta_prep(const b200_delta_inputs* inputs, float* q, float* k, float* v, float* beta,
                               float* log_decay, int64_t rows, int64_t sequences, int64_t longest, int dtype,
                               void* stream) {
  DeltaInputs p;
  if (!delta_inputs_from(inputs, &p) || !q || !k || !v || !beta || !log_decay || rows < 0 ||
      sequences < 0 || longest < 0)
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (rows > INT32_MAX) return B200_ERR_TOO_LARGE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_BF16 && (p.dim == 64 || p.dim == 128) && p.vdim == p.dim && p.taps <= 4 && longest >= 16 &&
      p.row_stride % 8 == 0 && p.gate_row_stride % 8 == 0 && p.q_column % 8 == 0 && p.k_column % 8 == 0 &&
      p.v_column % 8 == 0 && (p.decay_dim == 1 || (p.decay_column % 8 == 0 && aligned16(p.gates) && aligned16(p.dt_bias))) &&
      aligned16(p.input) && aligned16(p.ring) && sequences <= 65535) {
    const dim3 grid(static_cast<unsigned>(ceil_div(longest, 32)), static_cast<unsigned>(ceil_div(2 * p.kv_heads + 2 * p.heads, 8)),
                    static_cast<unsigned>(sequences));
    if (p.dim == 64) delta_prep_tiled_kernel<2><<<grid, 256, 0, s>>>(p, q, k, v, beta, log_decay);
    else delta_prep_tiled_kernel<4><<<grid, 256, 0, s>>>(p, q, k, v, beta, log_decay);
    return launch_status();
  }
  if (dtype == B200_F32)
    delta_prep_kernel<float><<<static_cast<unsigned>(rows), 256, 0, s>>>(p, q, k, v, beta, log_decay);
  else
    delta_prep_kernel<__nv_bfloat16><<<static_cast<unsigned>(rows), 256, 0, s>>>(p, q, k, v, beta, log_decay);
  return launch_status();
}

extern "C" int b200_conv_tail(const b200_delta_inputs* inputs, int64_t sequences, int dtype, void* stream) {
  DeltaInputs p;
  if (!delta_inputs_from(inputs, &p) || sequences < 0) return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (sequences == 0 || p.taps <= 1) return B200_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid(static_cast<unsigned>(sequences), static_cast<unsigned>(ceil_div(2 * p.kv_heads * p.dim + p.heads * p.vdim, 256)));
  if (dtype == B200_F32) conv_tail_kernel<float><<<grid, 256, 0, s>>>(p);
  else conv_tail_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(p);
  return launch_status();
}

extern "C" int b200_recurrence_scan(const float* q, const float* k, const float* v, const float* beta,
                                    const float* decay, float* state, float* output,
                                    const int32_t* token_sequence, const int32_t* starts, const int32_t* slots,
                                    const int32_t* bases, int64_t sequences, int64_t heads, int64_t kv_heads,
                                    int64_t dim, int64_t vdim, int64_t state_row, int64_t decay_dim, void* stream) {
  if (!q || !k || !v || !decay || !state || !output || !starts || !slots || !bases || sequences < 0 ||
      heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || dim <= 0 || vdim <= 0 || state_row < vdim ||
      (decay_dim != 1 && decay_dim != dim))
    return B200_ERR_BAD_ARGUMENT;
  if (sequences == 0) return B200_OK;
  if (sequences > 65535 || heads > 65535) return B200_ERR_TOO_LARGE;
  ScanParams p{q, k, v, beta, decay, state, output, {token_sequence, starts, slots, bases},
               static_cast<int>(heads), static_cast<int>(kv_heads), static_cast<int>(dim),
               static_cast<int>(vdim), static_cast<int>(state_row), static_cast<int>(decay_dim)};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return beta != nullptr ? dispatch_scan<true>(p, sequences, s) : dispatch_scan<false>(p, sequences, s);
}
