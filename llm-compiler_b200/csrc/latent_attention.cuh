// The split-KV form of latent attention on tcgen05 (latent_attention_tcgen05.cu), as latent_attention.cu
// calls it, and what the split kernels share.
#pragma once

#include "hybrid.cuh"

namespace b200 {

// The keys of split `split`: equal shares of at least 128 keys, in whole steps of `step`.
__device__ __forceinline__ void latent_split_range(int64_t keys, int splits, int split, int step, int64_t& begin,
                                                   int64_t& end) {
  int64_t share = (keys + splits - 1) / splits;
  if (share < 128) share = 128;
  share = (share + step - 1) / step * step;
  begin = share * split;
  end = begin + share < keys ? begin + share : keys;
}

struct LatentTcPlan {
  int n, pairs, ring, row_blocks, splits, smem;  // n 0: the sizes do not fit
};
LatentTcPlan plan_latent_tcgen05(int64_t sequences, int64_t longest, int64_t heads, int64_t rank, int64_t context);
int latent_attention_tcgen05(const LatentTcPlan& plan, const void* q, const void* cache, float* partial, float2* stats,
                             const SequenceBatch& batch, int64_t rows, int64_t sequences, int64_t heads, int64_t rank,
                             int64_t slots, int64_t capacity, double scale, int32_t* status, cudaStream_t stream);

}  // namespace b200
