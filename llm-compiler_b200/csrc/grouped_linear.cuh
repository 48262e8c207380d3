// Products of expert-sorted rows with a stack of weights, as experts.cu calls them.
#pragma once

#include "common.cuh"

namespace b200 {

struct GroupedLinearParams {
  const int32_t* tiles;  // [max_tiles][2]: expert (-1: none), rows held
  const float* scores;   // [sorted rows] or NULL (SwiGLU form only)
  void* out;             // [sorted rows, n], or [sorted rows, n / 2] with SwiGLU
  int32_t* clear;        // set to zero, or NULL
  int32_t* status;
  int clear_count, k, n, tile, max_tiles, experts, swiglu;
};

// bf16, k and the weight rows multiples of 8; tile a multiple of 16 up to 256
int grouped_linear_tcgen05(const GroupedLinearParams& p, const void* x, const void* w, cudaStream_t stream);

}  // namespace b200
