// Products of expert-sorted rows with a stack of weights, as experts.cu calls them.
#pragma once

#include "common.cuh"

namespace b200 {

struct GroupedLinearParams {
  const int32_t* tiles;  // [max_tiles][2]: expert (-1: none, and none behind it), rows held
  const int32_t* index;  // [sorted rows]: row of x, or NULL: x is sorted itself
  const float* scores;   // [sorted rows] or NULL (SwiGLU form only)
  void* out;             // [sorted rows, n], or [sorted rows, n / 2] with SwiGLU
  int32_t* status;
  int k, n, tile, max_tiles, x_rows, experts, swiglu;
};

// bf16, k and the weight rows multiples of 8; tile 16, 32, 64, 128 or 256; with an index at most tile rows of x
int grouped_linear_tcgen05(const GroupedLinearParams& p, const void* x, const void* w, cudaStream_t stream);

}  // namespace b200
