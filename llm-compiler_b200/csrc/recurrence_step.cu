// Decode step of the recurrent mixers, one token per sequence, in one launch: operand preparation
// (rotation, or short convolution, unit norm, decays and step size), state update, read-out, per-head
// RMS norm and output gate. One CTA per (head, sequence) holds the head's whole state in registers:
// it is read once and written once, 16 bytes per access, which is what the step costs.
//
// With the decayed state P = diag(g) S both products of the step come from one pass over it:
//   a = P^T k, b = P^T q;  u = beta (v - a) (delta) or v (retention);  o = b + (k . q) u;  S' = P + k u^T
#include "common.cuh"
#include "hybrid.cuh"
#include "recurrence.cuh"

namespace b200 {
namespace {

struct StepOutput {
  float* state;       // [slots, heads, dim, state_row]
  int state_row;      // a multiple of 4
  const void* gate;   // T [rows, gate_row_stride], head-major from column 0
  int64_t gate_row_stride;
  int gate_kind;
  const void* weight; // T [vdim] or NULL
  void* out;          // T [rows, out_row_stride], zeros behind heads * vdim
  int64_t out_row_stride;
  float eps;
  int early_state;    // the state may be read before the dependency wait
};

// `Inputs` is DeltaInputs or RetentionInputs. R: state rows per thread.
template <typename T, typename Inputs, int THREADS, int R>
__global__ void __launch_bounds__(THREADS) recurrence_step_kernel(const Inputs p, const StepOutput o) {
  constexpr bool kDelta = Inputs::kDelta;
  constexpr int kWarps = THREADS / 32;
  extern __shared__ float smem[];
  float* qs = smem;                    // [dim]
  float* ks = qs + p.dim;              // [dim]
  float* gs = ks + p.dim;              // [dim] decay of a key channel
  float* vs = gs + p.dim;              // [vdim]
  float* sums = smem + ((3 * p.dim + p.vdim + 3) & ~3);  // [2][row groups][state_row], 16-byte aligned
  __shared__ float partial[3][kWarps];
  grid_launch_dependents();
  const int head = blockIdx.x;
  const int64_t row = blockIdx.y;      // one row per sequence
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int columns = o.state_row / 4;
  const int groups = THREADS / columns;
  const int group = threadIdx.x / columns, column = (threadIdx.x % columns) * 4;
  const bool own = group < groups;
  if (!o.early_state) grid_dependency_wait_cta();
  const int slot = p.batch.slots[row];
  const int64_t position = p.batch.bases[row];
  T* out = static_cast<T*>(o.out) + row * o.out_row_stride + static_cast<int64_t>(head) * p.vdim;
  float* state = o.state + (static_cast<int64_t>(slot < 0 ? 0 : slot) * p.heads + head) * p.dim * o.state_row + column;
  float4 s[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = group + groups * i;
    s[i] = own && r < p.dim && slot >= 0 && position > 0
               ? __ldcs(reinterpret_cast<const float4*>(state + static_cast<int64_t>(r) * o.state_row))
               : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  if (o.early_state) grid_dependency_wait_cta();
  const T* gate = static_cast<const T*>(o.gate) + row * o.gate_row_stride + static_cast<int64_t>(head) * p.vdim;

  // ---- operands ----
  float beta = 0.0f;
  float q_squares = 0.0f, k_squares = 0.0f, along = 0.0f;  // sums over the key channels
  if (slot >= 0) {
    // (qs, ks, gs and vs lie side by side in the items' order)
    for (int item = threadIdx.x; item < 3 * p.dim + p.vdim; item += THREADS)
      qs[item] = step_operand<T>(p, head, item, row, position, slot);
    beta = step_beta<T>(p, row, head);
  }
  __syncthreads();
  if (slot >= 0) {
    for (int c = threadIdx.x; c < p.dim; c += THREADS) {
      const float q = qs[c], k = ks[c];
      q_squares += q * q;
      k_squares += k * k;
      along += q * k;
    }
  }
  q_squares = warp_sum(q_squares);
  k_squares = warp_sum(k_squares);
  along = warp_sum(along);
  if (lane == 0) {
    partial[0][warp] = q_squares;
    partial[1][warp] = k_squares;
    partial[2][warp] = along;
  }
  __syncthreads();
  if (slot < 0) {
    for (int c = threadIdx.x; c < p.vdim; c += THREADS) Elem<T>::store(out + c, 0.0f);
    return;
  }
  q_squares = k_squares = along = 0.0f;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) {
    q_squares += partial[0][w];
    k_squares += partial[1][w];
    along += partial[2][w];
  }
  // unit norms (delta) as factors of the products they enter
  const float q_factor = kDelta ? step_q_scale(p) / sqrtf(q_squares + kUnitEpsilon) : 1.0f;
  const float k_factor = kDelta ? 1.0f / sqrtf(k_squares + kUnitEpsilon) : 1.0f;

  // ---- one pass over the decayed state ----
  float4 a = make_float4(0.0f, 0.0f, 0.0f, 0.0f), b = a;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = group + groups * i;
    if (r < p.dim) {
      const float g = gs[r], k = ks[r], q = qs[r];
      s[i].x *= g; s[i].y *= g; s[i].z *= g; s[i].w *= g;
      if (kDelta) {
        a.x = fmaf(s[i].x, k, a.x); a.y = fmaf(s[i].y, k, a.y); a.z = fmaf(s[i].z, k, a.z); a.w = fmaf(s[i].w, k, a.w);
      }
      b.x = fmaf(s[i].x, q, b.x); b.y = fmaf(s[i].y, q, b.y); b.z = fmaf(s[i].z, q, b.z); b.w = fmaf(s[i].w, q, b.w);
    }
  }
  if (own) {
    if (kDelta) *reinterpret_cast<float4*>(sums + group * o.state_row + column) = a;
    *reinterpret_cast<float4*>(sums + (groups + group) * o.state_row + column) = b;
  }
  __syncthreads();
  float squares = 0.0f;
  for (int c = threadIdx.x; c < p.vdim; c += THREADS) {
    float pk = 0.0f, pq = 0.0f;
    for (int g = 0; g < groups; ++g) {
      if (kDelta) pk += sums[g * o.state_row + c];
      pq += sums[(groups + g) * o.state_row + c];
    }
    const float u = kDelta ? beta * (vs[c] - pk * k_factor) : vs[c];
    const float read = (pq + along * k_factor * u) * q_factor;
    vs[c] = u * k_factor;  // what a row of the state gets of k
    sums[c] = read;        // (row group 0 of `a`, column c: read by this thread only, above)
    squares += read * read;
  }
  squares = warp_sum(squares);
  if (lane == 0) partial[0][warp] = squares;
  __syncthreads();
  squares = 0.0f;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) squares += partial[0][w];
  const float factor = 1.0f / sqrtf(squares / p.vdim + o.eps);
  for (int c = threadIdx.x; c < p.vdim; c += THREADS) {
    float v = sums[c] * factor;
    if (o.weight != nullptr) v *= Elem<T>::load(static_cast<const T*>(o.weight) + c);
    Elem<T>::store(out + c, v * gate_value(Elem<T>::load(gate + c), o.gate_kind));
  }
  if (head == p.heads - 1) {
    T* row_out = static_cast<T*>(o.out) + row * o.out_row_stride;
    for (int64_t c = static_cast<int64_t>(p.heads) * p.vdim + threadIdx.x; c < o.out_row_stride; c += THREADS)
      Elem<T>::store(row_out + c, 0.0f);
  }

  // ---- state ----
  if (own) {
    float4 u;  // columns past vdim (the row's padding) stay zero
    u.x = column < p.vdim ? vs[column] : 0.0f;
    u.y = column + 1 < p.vdim ? vs[column + 1] : 0.0f;
    u.z = column + 2 < p.vdim ? vs[column + 2] : 0.0f;
    u.w = column + 3 < p.vdim ? vs[column + 3] : 0.0f;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int r = group + groups * i;
      if (r < p.dim) {
        const float k = ks[r];
        s[i].x = fmaf(k, u.x, s[i].x); s[i].y = fmaf(k, u.y, s[i].y);
        s[i].z = fmaf(k, u.z, s[i].z); s[i].w = fmaf(k, u.w, s[i].w);
        __stcs(reinterpret_cast<float4*>(state + static_cast<int64_t>(r) * o.state_row), s[i]);
      }
    }
  }
  keep_step_inputs<T, THREADS>(p, head, row, position, slot);
}

template <typename T, typename Inputs, int THREADS, int R>
int launch_step(const Inputs& p, const StepOutput& o, int64_t sequences, cudaStream_t stream) {
  const int groups = THREADS / (o.state_row / 4);
  const int smem = (3 * p.dim + p.vdim + 3 + 2 * groups * o.state_row) * static_cast<int>(sizeof(float));
  auto kernel = recurrence_step_kernel<T, Inputs, THREADS, R>;
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
    return B200_ERR_LAUNCH;
  const dim3 grid(static_cast<unsigned>(p.heads), static_cast<unsigned>(sequences));
  return launch_chained(kernel, grid, dim3(THREADS), smem, stream, p, o) == cudaSuccess ? launch_status()
                                                                                        : B200_ERR_LAUNCH;
}

// State rows a thread of a CTA of `threads` holds; 0: the layout does not fit
int rows_per_thread(int threads, int dim, int state_row) {
  const int groups = threads / (state_row / 4);
  return groups < 1 ? 0 : (dim + groups - 1) / groups;
}

template <typename T, typename Inputs>
int dispatch_step(const Inputs& p, const StepOutput& o, int64_t sequences, cudaStream_t stream) {
  const int r = rows_per_thread(256, p.dim, o.state_row);
  if (r >= 1 && r <= 2) return launch_step<T, Inputs, 256, 2>(p, o, sequences, stream);
  if (r >= 1 && r <= 4) return launch_step<T, Inputs, 256, 4>(p, o, sequences, stream);
  if (r >= 1 && r <= 8) return launch_step<T, Inputs, 256, 8>(p, o, sequences, stream);
  if (r >= 1 && r <= 16) return launch_step<T, Inputs, 256, 16>(p, o, sequences, stream);
  const int wide = rows_per_thread(512, p.dim, o.state_row);
  if (wide >= 1 && wide <= 16) return launch_step<T, Inputs, 512, 16>(p, o, sequences, stream);
  return B200_ERR_UNSUPPORTED;  // a state beyond 128 KB: prep, scan and gated norm as separate launches
}

template <typename Inputs>
int step(const Inputs& p, const b200_step_output* out, int64_t sequences, int dtype, void* stream) {
  if (!out || !out->state || !out->gate || !out->output || sequences < 0 || out->state_row < p.vdim ||
      out->state_row % 4 != 0 || (out->gate_kind != B200_GATE_SILU && out->gate_kind != B200_GATE_SIGMOID))
    return B200_ERR_BAD_ARGUMENT;
  if (dtype != B200_F32 && dtype != B200_BF16) return B200_ERR_UNSUPPORTED;
  if (sequences == 0) return B200_OK;
  if (sequences > 65535 || out->state_row > 2048) return B200_ERR_TOO_LARGE;
  if (!aligned16(out->state)) return B200_ERR_ALIGNMENT;
  StepOutput o{static_cast<float*>(out->state), static_cast<int>(out->state_row), out->gate, out->gate_row_stride,
               out->gate_kind, out->weight, out->output, out->output_row_stride, static_cast<float>(out->epsilon),
               (launch_mode() & B200_LAUNCH_STABLE_KV_PREFIX) != 0 ? 1 : 0};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == B200_F32 ? dispatch_step<float>(p, o, sequences, s)
                           : dispatch_step<__nv_bfloat16>(p, o, sequences, s);
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int b200_delta_step(const b200_delta_inputs* inputs, const b200_step_output* output, int64_t sequences,
                               int dtype, void* stream) {
  DeltaInputs p;
  if (!delta_inputs_from(inputs, &p)) return B200_ERR_BAD_ARGUMENT;
  return step(p, output, sequences, dtype, stream);
}

extern "C" int b200_retention_step(const b200_retention_inputs* inputs, const b200_step_output* output,
                                   int64_t sequences, int dtype, void* stream) {
  RetentionInputs p;
  if (!retention_inputs_from(inputs, &p) || !p.decay) return B200_ERR_BAD_ARGUMENT;
  return step(p, output, sequences, dtype, stream);
}
