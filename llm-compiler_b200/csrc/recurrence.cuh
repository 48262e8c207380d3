// Operands of the recurrent mixers as every kernel of theirs computes them (scan, decode step, chunked
// prefill): rotation, short causal convolution, decays and step sizes, all in fp32.
#pragma once

#include "hybrid.cuh"

namespace b200 {

constexpr float kUnitEpsilon = 1e-6f;  // inside the root of a unit norm

// cos / sin of position * base^(-2 i / dims). The product and its reduction to one turn are done in
// double, so that a far position costs no accuracy; the functions then see at most half a turn.
__device__ __forceinline__ void rotation_of(int64_t position, int i, int dims, double log2_base, float& c,
                                            float& s) {
  const double turns = static_cast<double>(position) * exp2(-2.0 * i / dims * log2_base) * 0.15915494309189535;
  sincospif(2.0f * static_cast<float>(turns - rint(turns)), &s, &c);
}

struct DeltaInputs {
  static constexpr bool kDelta = true;
  const void* input;   // T [rows, row_stride]: the projections of h
  const void* gates;   // T [rows, gate_row_stride]: decay columns [heads * decay_dim] from decay_column
  const void *q_conv, *k_conv, *v_conv;  // T [channels, taps] in time order
  const void* a_log;   // T [heads]
  const void* dt_bias; // T [heads * decay_dim]
  void* ring;          // T [slots, taps, 2 kv_heads dim + heads vdim]: inputs by position % taps
  SequenceBatch batch;
  int heads, kv_heads, dim, vdim, taps;
  int q_column, k_column, v_column, beta_column, decay_column;
  int64_t row_stride, gate_row_stride;
  float q_scale;
  int decay_dim;       // decays of a head: dim (one per key channel) or 1
};

inline bool delta_inputs_from(const b200_delta_inputs* in, DeltaInputs* out) {
  if (in == nullptr || !in->input || !in->gates || !in->q_conv || !in->k_conv || !in->v_conv || !in->a_log ||
      !in->dt_bias || !in->ring || !in->token_sequence || !in->starts || !in->slots || !in->bases ||
      in->heads <= 0 || in->kv_heads <= 0 || in->heads % in->kv_heads != 0 || in->dim <= 0 || in->vdim <= 0 ||
      in->taps <= 0 || (in->decay_dim != 1 && in->decay_dim != in->dim))
    return false;
  *out = DeltaInputs{in->input, in->gates, in->q_conv, in->k_conv, in->v_conv, in->a_log, in->dt_bias, in->ring,
                     {in->token_sequence, in->starts, in->slots, in->bases},
                     static_cast<int>(in->heads), static_cast<int>(in->kv_heads), static_cast<int>(in->dim),
                     static_cast<int>(in->vdim), static_cast<int>(in->taps), static_cast<int>(in->q_column),
                     static_cast<int>(in->k_column), static_cast<int>(in->v_column),
                     static_cast<int>(in->beta_column), static_cast<int>(in->decay_column), in->row_stride,
                     in->gate_row_stride, static_cast<float>(in->q_scale), static_cast<int>(in->decay_dim)};
  return true;
}

// Output of the short convolution of operand `which` (0 q, 1 k, 2 v), channel `channel`, for the token
// at `row` (the local-th of its portion, at `position`). Inputs of earlier portions come from the ring;
// before the start there are zeros.
template <typename T>
__device__ __forceinline__ float short_conv(const DeltaInputs& p, int which, int channel, int64_t row,
                                            int64_t local, int64_t position, int slot) {
  const T* taps = static_cast<const T*>(which == 0 ? p.q_conv : which == 1 ? p.k_conv : p.v_conv) +
                  static_cast<int64_t>(channel) * p.taps;
  const T* in = static_cast<const T*>(p.input) + row * p.row_stride +
                (which == 0 ? p.q_column : which == 1 ? p.k_column : p.v_column) + channel;
  const int qk = p.kv_heads * p.dim;
  const int channels = 2 * qk + p.heads * p.vdim;
  const T* ring = static_cast<const T*>(p.ring) + static_cast<int64_t>(slot) * p.taps * channels + which * qk + channel;
  const int entry = static_cast<int>(position) % p.taps;
  auto value_at = [&](int back) {
    const int index = entry - back < 0 ? entry - back + p.taps : entry - back;
    return back <= local ? Elem<T>::load(in - back * p.row_stride)
                         : Elem<T>::load(ring + static_cast<int64_t>(index) * channels);
  };
  const int reach = position < p.taps - 1 ? static_cast<int>(position) : p.taps - 1;
  float sum = 0.0f;
#pragma unroll
  for (int back = 0; back < 4; ++back)  // (the loads of the first four do not wait for one another)
    if (back <= reach) sum = fmaf(Elem<T>::load(taps + p.taps - 1 - back), value_at(back), sum);
  for (int back = 4; back <= reach; ++back) sum = fmaf(Elem<T>::load(taps + p.taps - 1 - back), value_at(back), sum);
  return sum;
}

template <typename T>
__device__ __forceinline__ float delta_beta(const DeltaInputs& p, int64_t row, int head) {
  return sigmoid_f32(Elem<T>::load(static_cast<const T*>(p.input) + row * p.row_stride + p.beta_column + head));
}

// log g of one key channel (of the head, where it has one decay)
template <typename T>
__device__ __forceinline__ float delta_log_decay(const DeltaInputs& p, int64_t row, int head, int c) {
  const int at = p.decay_dim == 1 ? head : head * p.dim + c;
  const float step = Elem<T>::load(static_cast<const T*>(p.gates) + row * p.gate_row_stride + p.decay_column + at) +
                     Elem<T>::load(static_cast<const T*>(p.dt_bias) + at);
  return -expf(Elem<T>::load(static_cast<const T*>(p.a_log) + head)) * softplus_f32(step);
}

struct RetentionInputs {
  static constexpr bool kDelta = false;
  const void* input;  // T [rows, row_stride]
  const float* decay; // [heads]
  SequenceBatch batch;
  int heads, dim, vdim, q_column, k_column, v_column, rot_dims;
  int64_t row_stride;
  double log2_base;   // log2 of the rotation base
  float k_scale;
};

inline bool retention_inputs_from(const b200_retention_inputs* in, RetentionInputs* out) {
  if (in == nullptr || !in->input || !in->token_sequence || !in->starts || !in->slots || !in->bases ||
      in->heads <= 0 || in->dim <= 0 || in->vdim <= 0 || in->rot_dims < 0 || in->rot_dims > in->dim ||
      in->rot_dims % 2 != 0 || in->rot_dims > 8192 || !(in->rot_base > 0.0))
    return false;
  *out = RetentionInputs{in->input, in->decay, {in->token_sequence, in->starts, in->slots, in->bases},
                         static_cast<int>(in->heads), static_cast<int>(in->dim), static_cast<int>(in->vdim),
                         static_cast<int>(in->q_column), static_cast<int>(in->k_column),
                         static_cast<int>(in->v_column), static_cast<int>(in->rot_dims), in->row_stride,
                         log2(in->rot_base), static_cast<float>(in->k_scale)};
  return true;
}

// ---- operands of a single decoded token, item by item: q [dim] and k [dim] (before a unit norm), decays
// [dim], v [vdim] of one head, in this order ----
template <typename T>
__device__ __forceinline__ float step_operand(const DeltaInputs& p, int head, int item, int64_t row, int64_t position,
                                              int slot) {
  if (item < 2 * p.dim) {
    const int which = item < p.dim ? 0 : 1;
    const int channel = head / (p.heads / p.kv_heads) * p.dim + item - which * p.dim;
    return silu_of(short_conv<T>(p, which, channel, row, 0, position, slot));
  }
  if (item < 3 * p.dim) return expf(delta_log_decay<T>(p, row, head, item - 2 * p.dim));
  return silu_of(short_conv<T>(p, 2, head * p.vdim + item - 3 * p.dim, row, 0, position, slot));
}
template <typename T>
__device__ __forceinline__ float step_operand(const RetentionInputs& p, int head, int item, int64_t row,
                                              int64_t position, int) {
  const T* in = static_cast<const T*>(p.input) + row * p.row_stride;
  if (item < 2 * p.dim) {
    const bool is_k = item >= p.dim;
    const int c = is_k ? item - p.dim : item;
    const T* src = in + (is_k ? p.k_column : p.q_column) + head * p.dim + c;
    float value = Elem<T>::load(src);
    const int half = p.rot_dims / 2;
    if (c < p.rot_dims) {
      const int other = c < half ? half : -half;
      float cosine, sine;
      rotation_of(position, c < half ? c : c - half, p.rot_dims, p.log2_base, cosine, sine);
      value = value * cosine + Elem<T>::load(src + other) * (c < half ? -sine : sine);
    }
    return is_k ? value * p.k_scale : value;
  }
  if (item < 3 * p.dim) return p.decay[head];
  return Elem<T>::load(in + p.v_column + head * p.vdim + item - 3 * p.dim);
}
template <typename T>
__device__ __forceinline__ float step_beta(const DeltaInputs& p, int64_t row, int head) {
  return delta_beta<T>(p, row, head);
}
template <typename T>
__device__ __forceinline__ float step_beta(const RetentionInputs&, int64_t, int) { return 1.0f; }
__device__ __forceinline__ float step_q_scale(const DeltaInputs& p) { return p.q_scale; }
__device__ __forceinline__ float step_q_scale(const RetentionInputs&) { return 1.0f; }

// This token's convolution inputs into the ring entry of its position, which no CTA of the step reads
// (the entries read are those of the taps - 1 positions before it).
template <typename T, int THREADS>
__device__ __forceinline__ void keep_step_inputs(const DeltaInputs& p, int head, int64_t row, int64_t position,
                                                 int slot) {
  if (p.taps <= 1) return;
  const int shared = p.heads / p.kv_heads, qk = p.kv_heads * p.dim;
  const int channels = 2 * qk + p.heads * p.vdim;
  T* ring = static_cast<T*>(p.ring) + (static_cast<int64_t>(slot) * p.taps + position % p.taps) * channels;
  const T* in = static_cast<const T*>(p.input) + row * p.row_stride;
  if (head % shared == 0) {
    const int first = head / shared * p.dim;
    for (int c = threadIdx.x; c < p.dim; c += THREADS) {
      ring[first + c] = in[p.q_column + first + c];
      ring[qk + first + c] = in[p.k_column + first + c];
    }
  }
  for (int c = threadIdx.x; c < p.vdim; c += THREADS)
    ring[2 * qk + head * p.vdim + c] = in[p.v_column + head * p.vdim + c];
}
template <typename T, int THREADS>
__device__ __forceinline__ void keep_step_inputs(const RetentionInputs&, int, int64_t, int64_t, int) {}

}  // namespace b200
