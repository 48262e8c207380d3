// What the kernels of the hybrid layers share: how the tokens of a step are cut into sequences, and
// the scalar functions of their gates and decays (fp32).
#pragma once

#include "common.cuh"

namespace b200 {

// The tokens of a step side by side: sequence s owns rows starts[s] .. starts[s + 1] - 1, lives in
// state slot slots[s] (-1: an idle row, nothing of it is read or kept) and its first row stands at
// position bases[s]. token_sequence[row] is the sequence of a row.
struct SequenceBatch {
  const int32_t* token_sequence;
  const int32_t* starts;
  const int32_t* slots;
  const int32_t* bases;
  __device__ __forceinline__ int64_t position(int sequence, int64_t row) const {
    return static_cast<int64_t>(bases[sequence]) + (row - starts[sequence]);
  }
};

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_of(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float gate_value(float x, int kind) {
  return kind == B200_GATE_SILU ? silu_of(x) : sigmoid_f32(x);
}

}  // namespace b200
