// Chunked form of the linear recurrences for prompts: 64 tokens at a time become matrix products.
//
// With P_i the product of the decays of a chunk's tokens 0 .. i (per key channel), S the state in front
// of the chunk and all products per channel,
//   u_i = beta_i (v_i - (P_i k_i)^T S - sum_{j<i} [k_i . (P_i / P_j) k_j] u_j)       (delta; retention: u_i = v_i)
//   o_i = (P_i q_i)^T S + sum_{j<=i} [q_i . (P_i / P_j) k_j] u_j
//   S'  = P_last S + sum_j ((P_last / P_j) k_j) u_j^T
// The first kernel does everything that does not need S, for all chunks at once: the two triangular
// matrices, the triangular solve that turns u into u0 - W S, and the decayed operands. The second walks
// the chunks of a sequence with a slice of S's columns in registers.
//
// Precision: decays stay logarithms until they are differences of one sign (products of decays are taken
// as sums over the tokens between, never as quotients), the triangular solve is fp32, and every product
// on the tensor cores splits its fp32 operands into two bf16 numbers (hi hi + hi lo + lo hi), which keeps
// 16 bits of mantissa. Within 16 tokens the decayed products are built up token by token instead. Where a
// head has one decay, P_i / P_j is a factor of the plain product k_i . k_j: 2 to a difference of running
// sums, which are kept in double.
#include "common.cuh"
#include "hybrid.cuh"

namespace b200 {
namespace {

constexpr int kChunk = 64, kSub = 16, kSubs = kChunk / kSub;
constexpr int kIntraThreads = 512;
template <int N>
struct IntConstant { static constexpr int value = N; };

struct ChunkParams {
  const float *q, *k, *v;   // [rows, kv_heads, dim] x 2, [rows, heads, vdim]
  const float* beta;        // [rows, heads] (delta)
  const float* decay;       // log g [rows, heads, dim] or [rows, heads] (delta); decay [heads] (retention)
  float* state;             // [slots, heads, dim, state_row]
  float* output;            // [rows, heads, vdim]
  SequenceBatch batch;
  const int32_t* chunk_starts;  // [sequences + 1]
  int sequences, heads, kv_heads, dim, vdim, state_row;
  unsigned char* workspace;
};

// What the first kernel leaves per (chunk, head): operand planes [64][D] of bf16, high then low parts.
template <int D>
struct ChunkLayout {
  static constexpr int64_t kPlane = kChunk * D * 2, kSquare = kChunk * kChunk * 2;
  static constexpr int64_t kQ = 0, kK = 2 * kPlane, kA = 4 * kPlane, kEnd = kA + 2 * kSquare, kLast = kEnd + D * 4;
  static constexpr int64_t kW = kLast;                       // delta only
  static constexpr int64_t kU = kW + 2 * kPlane;             // fp32 [64][vdim rounded up to 32], delta only
  __host__ __device__ static int64_t bytes(bool delta, int vdim) {
    return delta ? kU + static_cast<int64_t>(kChunk) * ((vdim + 31) / 32 * 32) * 4 : kLast;
  }
};

__device__ __forceinline__ void split_bf16x2(float a, float b, uint32_t& high, uint32_t& low) {
  high = pack_bf16x2(a, b);
  low = pack_bf16x2(a - bf16_lo(high), b - bf16_hi(high));
}

// ---- within the chunks -------------------------------------------------------------------
constexpr int kTriangle = kChunk + 8;  // row pitch (bf16) of the solve's triangular planes
constexpr int kInverse = kSub + 8;     // of the inverted 16 x 16 blocks

template <int D>
constexpr int intra_smem_bytes() {
  constexpr int blocks = (2 * kSub + (kSubs - 1) * kSub) * 2 * (D + 8) * 2;
  constexpr int solve = 2 * kChunk * kTriangle * 2 + 2 * kChunk * kInverse * 2;
  return 4 * kChunk * (D + 4) * 4 + 2 * kChunk * (kChunk + 4) * 4 + 2 * kSubs * D * 4 + (blocks > solve ? blocks : solve);
}

// Which sequence a chunk belongs to, its first row and how many of its 64 rows exist.
__device__ __forceinline__ int locate_chunk(const ChunkParams& p, int chunk, int64_t& row0) {
  int sequence = 0;
  while (sequence + 1 < p.sequences && p.chunk_starts[sequence + 1] <= chunk) ++sequence;
  row0 = p.batch.starts[sequence] + static_cast<int64_t>(chunk - p.chunk_starts[sequence]) * kChunk;
  const int64_t left = p.batch.starts[sequence + 1] - row0;
  return left < kChunk ? static_cast<int>(left) : kChunk;
}

__device__ __forceinline__ float4 exp2_4(float4 x) {
  return make_float4(exp2f(x.x), exp2f(x.y), exp2f(x.z), exp2f(x.w));
}
__device__ __forceinline__ float4 mul4(float4 a, float4 b) {
  return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w);
}
__device__ __forceinline__ float4 add4(float4 a, float4 b) {
  return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w);
}
__device__ __forceinline__ float dot4(float4 a, float4 b) {
  return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, a.w * b.w)));
}
__device__ __forceinline__ void split4(float4 v, uint2& high, uint2& low) {
  split_bf16x2(v.x, v.y, high.x, low.x);
  split_bf16x2(v.z, v.w, high.y, low.y);
}
// Four channels of a row of an operand; zeros outside
__device__ __forceinline__ float4 load4(const float* source, int c, int dim, bool inside, bool whole) {
  float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  if (inside && whole) return *reinterpret_cast<const float4*>(source + c);
  if (inside) {
    if (c < dim) v.x = source[c];
    if (c + 1 < dim) v.y = source[c + 1];
    if (c + 2 < dim) v.z = source[c + 2];
    if (c + 3 < dim) v.w = source[c + 3];
  }
  return v;
}

// Triangular solve (I + lower) [W | U] = beta [P k | v] on the tensor cores, transposed: a warp owns 16
// columns, Y_I = (R_I - sum_{J<I} Y_J lower_IJ^T) inverse_I^T stays in its registers throughout.
// triangle: [2][64][kTriangle] planes of minus the blocks below the diagonal; inverse: [2][64][kInverse]
// inverted diagonal blocks; decayed_key(i, c): entry c of P_i k_i; staging: [2][64][D] planes of W.
template <int D, typename DecayedKey>
__device__ __forceinline__ void solve_chunk(const ChunkParams& p, const __nv_bfloat16* triangle,
                                            const __nv_bfloat16* inverse, const float* betas, __nv_bfloat16* staging,
                                            unsigned char* out, int64_t row0, int count, int head, int warp, int lane,
                                            DecayedKey decayed_key) {
  using Layout = ChunkLayout<D>;
  const int v_row = (p.vdim + 31) / 32 * 32;
  for (int tile = warp; tile < (D + v_row) / 16; tile += blockDim.x / 32) {
    const int c0 = tile * 16 + (lane >> 2);  // fragment rows c0 and c0 + 8 are columns of [W | U]
    float rhs[kSubs][2][4];
#pragma unroll
    for (int I = 0; I < kSubs; ++I)
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = I * kSub + h * 8 + (lane & 3) * 2 + (e & 1), c = c0 + (e >> 1) * 8;
          if (tile < D / 16) {
            rhs[I][h][e] = betas[i] * decayed_key(i, c);
          } else {
            const int vc = c - D;
            rhs[I][h][e] = i < count && vc < p.vdim ? p.v[((row0 + i) * p.heads + head) * p.vdim + vc] : 0.0f;
          }
        }
    uint32_t yh[kSubs][4], yl[kSubs][4];
#pragma unroll
    for (int I = 0; I < kSubs; ++I) {
      float acc[2][4];
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          acc[h][e] = tile < D / 16 ? rhs[I][h][e] : rhs[I][h][e] * betas[I * kSub + h * 8 + (lane & 3) * 2 + (e & 1)];
      const int n_row = I * kSub + ((lane >> 4) << 3) + (lane & 7), k_half = ((lane >> 3) & 1) * 8;
      auto multiply = [&](const uint32_t (&ah)[4], const uint32_t (&al)[4], const __nv_bfloat16* plane, int pitch,
                          int column, float (&to)[2][4]) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4(bh, smem_u32(plane + n_row * pitch + column + k_half));
        ldmatrix_x4(bl, smem_u32(plane + (kChunk + n_row) * pitch + column + k_half));
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          mma_bf16_16816(to[h], ah, bh[h * 2], bh[h * 2 + 1]);
          mma_bf16_16816(to[h], ah, bl[h * 2], bl[h * 2 + 1]);
          mma_bf16_16816(to[h], al, bh[h * 2], bh[h * 2 + 1]);
        }
      };
#pragma unroll
      for (int J = 0; J < I; ++J) multiply(yh[J], yl[J], triangle, kTriangle, J * kSub, acc);
      uint32_t zh[4], zl[4];
      split_bf16x2(acc[0][0], acc[0][1], zh[0], zl[0]);
      split_bf16x2(acc[0][2], acc[0][3], zh[1], zl[1]);
      split_bf16x2(acc[1][0], acc[1][1], zh[2], zl[2]);
      split_bf16x2(acc[1][2], acc[1][3], zh[3], zl[3]);
      float y[2][4] = {};
      multiply(zh, zl, inverse, kInverse, 0, y);
      split_bf16x2(y[0][0], y[0][1], yh[I][0], yl[I][0]);
      split_bf16x2(y[0][2], y[0][3], yh[I][1], yl[I][1]);
      split_bf16x2(y[1][0], y[1][1], yh[I][2], yl[I][2]);
      split_bf16x2(y[1][2], y[1][3], yh[I][3], yl[I][3]);
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = I * kSub + h * 8 + (lane & 3) * 2 + (e & 1), c = c0 + (e >> 1) * 8;
          if (tile < D / 16) {
            const __nv_bfloat16 high = __float2bfloat16_rn(y[h][e]);
            staging[i * D + c] = high;
            staging[(kChunk + i) * D + c] = __float2bfloat16_rn(y[h][e] - __bfloat162float(high));
          } else {
            reinterpret_cast<float*>(out + Layout::kU)[i * v_row + c - D] = y[h][e];
          }
        }
    }
  }
  __syncthreads();
  for (int item = threadIdx.x; item < 2 * kChunk * D / 8; item += blockDim.x)
    reinterpret_cast<uint4*>(out + Layout::kW)[item] = reinterpret_cast<const uint4*>(staging)[item];
}

// (I + N)^-1 of the 16 x 16 diagonal blocks, one column a thread of the CTA's last 64
__device__ __forceinline__ void invert_diagonal_blocks(const float* lower, int pitch, __nv_bfloat16* inverse) {
  if (threadIdx.x < blockDim.x - kChunk) return;
  const int column = threadIdx.x - (blockDim.x - kChunk), block = column / kSub * kSub, own = column % kSub;
  float x[kSub];
#pragma unroll
  for (int i = 0; i < kSub; ++i) {
    float v = i == own ? 1.0f : 0.0f;
#pragma unroll
    for (int j = 0; j < i; ++j) v = fmaf(-lower[(block + i) * pitch + block + j], x[j], v);
    x[i] = v;
    const __nv_bfloat16 high = __float2bfloat16_rn(v);
    inverse[(block + i) * kInverse + own] = high;
    inverse[(kChunk + block + i) * kInverse + own] = __float2bfloat16_rn(v - __bfloat162float(high));
  }
}

// Retention: one decay per head, so the decayed products are the plain ones times decay^(i - j).
template <int D>
__global__ void __launch_bounds__(kIntraThreads) chunk_intra_retention_kernel(const ChunkParams p) {
  constexpr int PB = (D + 8) * 2;
  using Layout = ChunkLayout<D>;
  extern __shared__ __align__(128) unsigned char smem[];
  unsigned char* q_planes = smem;                          // [2][64][PB]
  unsigned char* k_planes = smem + 2 * kChunk * PB;
  const int chunk = blockIdx.x, head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int64_t row0;
  const int count = locate_chunk(p, chunk, row0);
  const int kv_head = head / (p.heads / p.kv_heads);
  unsigned char* out = p.workspace + (static_cast<int64_t>(chunk) * p.heads + head) * Layout::bytes(false, p.vdim);
  const float decay = fmaxf(log2f(p.decay[head]), -126.0f);  // (less than 2^-126 is nothing)
  const bool whole = p.dim == D;
#pragma unroll
  for (int i = 0; i < kChunk * D / 4 / kIntraThreads; ++i) {
    const int item = threadIdx.x + i * kIntraThreads, t = item / (D / 4), c = item % (D / 4) * 4;
    const int64_t source = ((row0 + t) * p.kv_heads + kv_head) * p.dim;
    const float4 q = load4(p.q + source, c, p.dim, t < count, whole), k = load4(p.k + source, c, p.dim, t < count, whole);
    const float into = exp2f(decay * (t + 1)), rest = t < count ? exp2f(decay * (count - 1 - t)) : 0.0f;
    uint2 high, low;
    split4(q, high, low);
    *reinterpret_cast<uint2*>(q_planes + t * PB + c * 2) = high;
    *reinterpret_cast<uint2*>(q_planes + (kChunk + t) * PB + c * 2) = low;
    split4(k, high, low);
    *reinterpret_cast<uint2*>(k_planes + t * PB + c * 2) = high;
    *reinterpret_cast<uint2*>(k_planes + (kChunk + t) * PB + c * 2) = low;
    split4(mul4(q, make_float4(into, into, into, into)), high, low);
    reinterpret_cast<uint2*>(out + Layout::kQ)[item] = high;
    reinterpret_cast<uint2*>(out + Layout::kQ + Layout::kPlane)[item] = low;
    split4(mul4(k, make_float4(rest, rest, rest, rest)), high, low);
    reinterpret_cast<uint2*>(out + Layout::kK)[item] = high;
    reinterpret_cast<uint2*>(out + Layout::kK + Layout::kPlane)[item] = low;
  }
  if (threadIdx.x < D) reinterpret_cast<float*>(out + Layout::kEnd)[threadIdx.x] = exp2f(decay * count);
  __syncthreads();
  // 16 warps: 16 rows x 16 columns each
  const int m0 = (warp >> 2) * 16, n0 = (warp & 3) * 16;
  float acc[2][4] = {};
  if (n0 <= m0) {
    const uint32_t a_base = smem_u32(q_planes) + (m0 + (lane & 15)) * PB + (lane >> 4) * 16;
    const uint32_t b_base = smem_u32(k_planes) + (n0 + ((lane >> 4) << 3) + (lane & 7)) * PB + ((lane >> 3) & 1) * 16;
#pragma unroll
    for (int step = 0; step < D / 16; ++step) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      ldmatrix_x4(ah, a_base + step * 32);
      ldmatrix_x4(al, a_base + kChunk * PB + step * 32);
      ldmatrix_x4(bh, b_base + step * 32);
      ldmatrix_x4(bl, b_base + kChunk * PB + step * 32);
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        mma_bf16_16816(acc[h], ah, bh[h * 2], bh[h * 2 + 1]);
        mma_bf16_16816(acc[h], ah, bl[h * 2], bl[h * 2 + 1]);
        mma_bf16_16816(acc[h], al, bh[h * 2], bh[h * 2 + 1]);
      }
    }
  }
#pragma unroll
  for (int h = 0; h < 2; ++h)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = m0 + (lane >> 2) + half * 8, j = n0 + h * 8 + (lane & 3) * 2;
      const float a = i >= j ? acc[h][half * 2] * exp2f(decay * (i - j)) : 0.0f;
      const float b = i >= j + 1 ? acc[h][half * 2 + 1] * exp2f(decay * (i - j - 1)) : 0.0f;
      uint32_t high, low;
      split_bf16x2(a, b, high, low);
      reinterpret_cast<uint32_t*>(out + Layout::kA)[(i * kChunk + j) / 2] = high;
      reinterpret_cast<uint32_t*>(out + Layout::kA + Layout::kSquare)[(i * kChunk + j) / 2] = low;
    }
}

// The delta rule with one decay per head: both triangular matrices are plain products times 2^(x_i - x_j),
// x the running sum of log2 g.
template <int D>
constexpr int intra_head_delta_smem_bytes() {
  return 4 * kChunk * (D + 8) * 2 + kChunk * (kChunk + 4) * 4 + 2 * kChunk * kTriangle * 2 + 2 * kChunk * kInverse * 2;
}
constexpr int kHeadDeltaThreads = 256;  // two CTAs per SM: one's loads and solve under the other's products
template <int D>
__global__ void __launch_bounds__(kHeadDeltaThreads, 2) chunk_intra_head_delta_kernel(const ChunkParams p) {
  constexpr int PM = kChunk + 4, PB = (D + 8) * 2;
  using Layout = ChunkLayout<D>;
  extern __shared__ __align__(128) unsigned char smem[];
  unsigned char* q_planes = smem;                          // [2][64][PB], later the staging of W's planes
  unsigned char* k_planes = smem + 2 * kChunk * PB;
  float* lower = reinterpret_cast<float*>(k_planes + 2 * kChunk * PB);  // [64][PM]
  __nv_bfloat16* triangle = reinterpret_cast<__nv_bfloat16*>(lower + kChunk * PM);
  __nv_bfloat16* inverse = triangle + 2 * kChunk * kTriangle;
  __shared__ float betas[kChunk], into[kChunk];   // into: 2^x
  __shared__ double sums[kChunk];                 // x
  const int chunk = blockIdx.x, head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int64_t row0;
  const int count = locate_chunk(p, chunk, row0);
  const int kv_head = head / (p.heads / p.kv_heads);
  unsigned char* out = p.workspace + (static_cast<int64_t>(chunk) * p.heads + head) * Layout::bytes(true, p.vdim);
  const bool whole = p.dim == D;
  constexpr int kRounds = kChunk * D / 4 / kHeadDeltaThreads;
  // (the queries' loads are in flight while the decays are summed up, the keys' while the queries are split)
  auto load_rows = [&](const float* from, float4* rows) {
#pragma unroll
    for (int i = 0; i < kRounds; ++i) {
      const int item = threadIdx.x + i * kHeadDeltaThreads, t = item / (D / 4), c = item % (D / 4) * 4;
      rows[i] = load4(from + ((row0 + t) * p.kv_heads + kv_head) * p.dim, c, p.dim, t < count, whole);
    }
  };
  float4 q[kRounds], k[kRounds];
  load_rows(p.q, q);
  if (warp == 0) {  // two tokens a lane
    double x[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = lane * 2 + e;
      const int64_t unit = (row0 + t) * p.heads + head;
      betas[t] = t < count ? p.beta[unit] : 0.0f;
      // (a token that keeps less than 2^-126 keeps nothing)
      x[e] = t < count ? static_cast<double>(fmaxf(p.decay[unit] * 1.4426950408889634f, -126.0f)) : 0.0;
    }
    x[1] += x[0];
    double total = x[1];
#pragma unroll
    for (int o = 1; o < 32; o *= 2) {
      const double before = __shfl_up_sync(0xffffffffu, total, o);
      if (lane >= o) total += before;
    }
    const double front = total - x[1];
    sums[lane * 2] = front + x[0];
    sums[lane * 2 + 1] = total;
    into[lane * 2] = exp2f(static_cast<float>(front + x[0]));
    into[lane * 2 + 1] = exp2f(static_cast<float>(total));
  }
  __syncthreads();
  const double end = sums[kChunk - 1];
  load_rows(p.k, k);
  auto split_rows = [&](const float4* rows, unsigned char* planes, unsigned char* decayed, auto factor) {
#pragma unroll
    for (int i = 0; i < kRounds; ++i) {
      const int item = threadIdx.x + i * kHeadDeltaThreads, t = item / (D / 4), c = item % (D / 4) * 4;
      const float f = factor(t);
      uint2 high, low;
      split4(rows[i], high, low);
      *reinterpret_cast<uint2*>(planes + t * PB + c * 2) = high;
      *reinterpret_cast<uint2*>(planes + (kChunk + t) * PB + c * 2) = low;
      split4(mul4(rows[i], make_float4(f, f, f, f)), high, low);
      reinterpret_cast<uint2*>(decayed)[item] = high;
      reinterpret_cast<uint2*>(decayed + Layout::kPlane)[item] = low;
    }
  };
  split_rows(q, q_planes, out + Layout::kQ, [&](int t) { return into[t]; });
  split_rows(k, k_planes, out + Layout::kK, [&](int t) { return exp2f(static_cast<float>(end - sums[t])); });
  if (threadIdx.x < D) reinterpret_cast<float*>(out + Layout::kEnd)[threadIdx.x] = into[kChunk - 1];
  __syncthreads();
  // 16 x 16 tiles of K K^T and of Q K^T: the ten on and below the diagonal, then zeros above it
  constexpr int kWarps = kHeadDeltaThreads / 32;
  for (int tile = warp; tile < 16; tile += kWarps) {
    int m = 0, n = tile;  // row by row below the diagonal; the last six above it
    if (tile < 10) {
      while (n > m) n -= ++m;
    } else {
      n = tile - 10;
      while (n >= 3 - m) n -= 3 - m++;
      n += m + 1;
    }
    const int m0 = m * 16, n0 = n * 16;
    float kk[2][4] = {}, qk[2][4] = {};
    if (n0 <= m0) {
      const uint32_t row_lane = (m0 + (lane & 15)) * PB + (lane >> 4) * 16;
      const uint32_t ka_base = smem_u32(k_planes) + row_lane, qa_base = smem_u32(q_planes) + row_lane;
      const uint32_t b_base = smem_u32(k_planes) + (n0 + ((lane >> 4) << 3) + (lane & 7)) * PB + ((lane >> 3) & 1) * 16;
#pragma unroll
      for (int step = 0; step < D / 16; ++step) {
        uint32_t kh[4], kl[4], qh[4], ql[4], bh[4], bl[4];
        ldmatrix_x4(kh, ka_base + step * 32);
        ldmatrix_x4(kl, ka_base + kChunk * PB + step * 32);
        ldmatrix_x4(qh, qa_base + step * 32);
        ldmatrix_x4(ql, qa_base + kChunk * PB + step * 32);
        ldmatrix_x4(bh, b_base + step * 32);
        ldmatrix_x4(bl, b_base + kChunk * PB + step * 32);
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          mma_bf16_16816(kk[h], kh, bh[h * 2], bh[h * 2 + 1]);
          mma_bf16_16816(qk[h], qh, bh[h * 2], bh[h * 2 + 1]);
          mma_bf16_16816(kk[h], kh, bl[h * 2], bl[h * 2 + 1]);
          mma_bf16_16816(qk[h], qh, bl[h * 2], bl[h * 2 + 1]);
          mma_bf16_16816(kk[h], kl, bh[h * 2], bh[h * 2 + 1]);
          mma_bf16_16816(qk[h], ql, bh[h * 2], bh[h * 2 + 1]);
        }
      }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = m0 + (lane >> 2) + half * 8, j = n0 + h * 8 + (lane & 3) * 2;
        float a[2], l[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float f = i >= j + e ? exp2f(static_cast<float>(sums[i] - sums[j + e])) : 0.0f;
          a[e] = qk[h][half * 2 + e] * f;
          l[e] = i > j + e ? kk[h][half * 2 + e] * f * betas[i] : 0.0f;
        }
        uint32_t high, low;
        split_bf16x2(a[0], a[1], high, low);
        reinterpret_cast<uint32_t*>(out + Layout::kA)[(i * kChunk + j) / 2] = high;
        reinterpret_cast<uint32_t*>(out + Layout::kA + Layout::kSquare)[(i * kChunk + j) / 2] = low;
        if (n0 == m0) *reinterpret_cast<float2*>(lower + i * PM + j) = make_float2(l[0], l[1]);
        if (n0 < m0) {
          split_bf16x2(-l[0], -l[1], high, low);
          *reinterpret_cast<uint32_t*>(triangle + i * kTriangle + j) = high;
          *reinterpret_cast<uint32_t*>(triangle + (kChunk + i) * kTriangle + j) = low;
        }
      }
  }
  __syncthreads();
  invert_diagonal_blocks(lower, PM, inverse);
  __syncthreads();
  const __nv_bfloat16* keys = reinterpret_cast<const __nv_bfloat16*>(k_planes);
  solve_chunk<D>(p, triangle, inverse, betas, reinterpret_cast<__nv_bfloat16*>(q_planes), out, row0, count, head, warp,
                 lane, [&](int i, int c) {
                   return (__bfloat162float(keys[i * (D + 8) + c]) + __bfloat162float(keys[(kChunk + i) * (D + 8) + c])) *
                          into[i];
                 });
}

template <int D>
__global__ void __launch_bounds__(kIntraThreads, 1) chunk_intra_delta_kernel(const ChunkParams p) {
  constexpr int PD = D + 4, PM = kChunk + 4, PB = (D + 8) * 2;  // pitches: floats, floats, bytes
  constexpr int kRounds = kChunk * D / 4 / kIntraThreads;        // float4 items of a [64][D] array per thread
  using Layout = ChunkLayout<D>;
  extern __shared__ __align__(128) unsigned char smem[];
  float* ks = reinterpret_cast<float*>(smem);       // [64][PD]
  float* qs = ks + kChunk * PD;                     // later the staging of W's planes
  float* xs = qs + kChunk * PD;                     // log2 g, later its running sum within 16 tokens
  float* gs = xs + kChunk * PD;                     // g, later the sum of log2 g over the rest of the 16 tokens
  float* lower = gs + kChunk * PD;                  // [64][PM] beta_i k_i . (P_i / P_j) k_j, j < i
  float* mixed = lower + kChunk * PM;               // [64][PM] q_i . (P_i / P_j) k_j, j <= i
  float* pre = mixed + kChunk * PM;                 // [4][D] log2 of the decay in front of 16 tokens
  float* post = pre + kSubs * D;                    // [4][D] ... behind them
  unsigned char* planes = reinterpret_cast<unsigned char*>(post + kSubs * D);
  __shared__ float betas[kChunk];
  const int chunk = blockIdx.x, head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int64_t row0;
  const int count = locate_chunk(p, chunk, row0);
  const int kv_head = head / (p.heads / p.kv_heads);
  unsigned char* out = p.workspace + (static_cast<int64_t>(chunk) * p.heads + head) * Layout::bytes(true, p.vdim);
  const bool whole = p.dim == D;
  {
    float4 k[kRounds], q[kRounds], x[kRounds];
#pragma unroll
    for (int i = 0; i < kRounds; ++i) {
      const int item = threadIdx.x + i * kIntraThreads, t = item / (D / 4), c = item % (D / 4) * 4;
      const int64_t source = ((row0 + t) * p.kv_heads + kv_head) * p.dim;
      k[i] = load4(p.k + source, c, p.dim, t < count, whole);
      q[i] = load4(p.q + source, c, p.dim, t < count, whole);
      x[i] = load4(p.decay + ((row0 + t) * p.heads + head) * p.dim, c, p.dim, t < count, whole);
    }
    if (threadIdx.x < kChunk)
      betas[threadIdx.x] = threadIdx.x < count ? p.beta[(row0 + threadIdx.x) * p.heads + head] : 0.0f;
    for (int item = threadIdx.x; item < kChunk * PM / 4; item += kIntraThreads)
      reinterpret_cast<float4*>(mixed)[item] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    constexpr float kLog2e = 1.4426950408889634f;
#pragma unroll
    for (int i = 0; i < kRounds; ++i) {
      const int item = threadIdx.x + i * kIntraThreads, at = item / (D / 4) * PD + item % (D / 4) * 4;
      // (a token that keeps less than 2^-126 keeps nothing)
      const float4 l = make_float4(fmaxf(x[i].x * kLog2e, -126.0f), fmaxf(x[i].y * kLog2e, -126.0f),
                                   fmaxf(x[i].z * kLog2e, -126.0f), fmaxf(x[i].w * kLog2e, -126.0f));
      *reinterpret_cast<float4*>(ks + at) = k[i];
      *reinterpret_cast<float4*>(qs + at) = q[i];
      *reinterpret_cast<float4*>(xs + at) = l;
      *reinterpret_cast<float4*>(gs + at) = exp2_4(l);
    }
  }
  __syncthreads();

  // ---- the 16 x 16 blocks on the diagonal: w = (P_i / P_j) k_j built up token by token ----
  // D / 4 lanes share four columns j of a block, four channels each; their eight sums per row are
  // reduced together, every exchange halving the number of sums a lane still carries.
  constexpr int LG = D / 4;
  if (static_cast<int>(threadIdx.x) / LG < 16) {
    const int group = threadIdx.x / LG, l = threadIdx.x % LG;
    const int block = group / 4 * kSub, j0 = group % 4 * 4;
    float4 w[4];
#pragma unroll
    for (int jj = 0; jj < 4; ++jj) w[jj] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    for (int i = 0; i < kSub; ++i) {
      const int at = (block + i) * PD + l * 4;
      const float4 kk = *reinterpret_cast<const float4*>(ks + at);
      const float4 qq = *reinterpret_cast<const float4*>(qs + at);
      const float4 gg = *reinterpret_cast<const float4*>(gs + at);
      float v[8];
#pragma unroll
      for (int jj = 0; jj < 4; ++jj) {
        w[jj] = i == j0 + jj ? kk : mul4(w[jj], gg);
        v[jj] = dot4(kk, w[jj]);
        v[4 + jj] = dot4(qq, w[jj]);
      }
      const bool is_q = (l & (LG / 2)) != 0, second = (l & (LG / 4)) != 0, odd = (l & (LG / 8)) != 0;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float received = __shfl_xor_sync(0xffffffffu, is_q ? v[e] : v[4 + e], LG / 2);
        v[e] = (is_q ? v[4 + e] : v[e]) + received;
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float received = __shfl_xor_sync(0xffffffffu, second ? v[e] : v[2 + e], LG / 4);
        v[e] = (second ? v[2 + e] : v[e]) + received;
      }
      const float received = __shfl_xor_sync(0xffffffffu, odd ? v[0] : v[1], LG / 8);
      float sum = (odd ? v[1] : v[0]) + received;
#pragma unroll
      for (int o = LG / 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      if ((l & (LG / 8 - 1)) == 0) {
        const int j = j0 + (second ? 2 : 0) + (odd ? 1 : 0), at_m = (block + i) * PM + block + j;
        if (is_q) mixed[at_m] = i >= j ? sum : 0.0f;
        else lower[at_m] = i > j ? sum * betas[block + i] : 0.0f;
      }
    }
  }
  __syncthreads();
  // ---- running sums of log2 g within 16 tokens, forwards (inclusive) and backwards (exclusive) ----
  for (int item = threadIdx.x; item < kSubs * D; item += kIntraThreads) {
    const int at = item / D * kSub * PD + item % D;
    float x[kSub];
#pragma unroll
    for (int i = 0; i < kSub; ++i) x[i] = xs[at + i * PD];
    float sum = 0.0f;
#pragma unroll
    for (int i = kSub - 1; i >= 0; --i) {
      gs[at + i * PD] = sum;
      sum += x[i];
    }
    sum = 0.0f;
#pragma unroll
    for (int i = 0; i < kSub; ++i) {
      sum += x[i];
      xs[at + i * PD] = sum;
    }
  }
  __syncthreads();
  for (int c = threadIdx.x; c < D; c += kIntraThreads) {
    float total[kSubs], sum = 0.0f;
#pragma unroll
    for (int s = 0; s < kSubs; ++s) {
      total[s] = xs[(s * kSub + kSub - 1) * PD + c];
      pre[s * D + c] = sum;
      sum += total[s];
    }
    reinterpret_cast<float*>(out + Layout::kEnd)[c] = exp2f(sum);
    sum = 0.0f;
#pragma unroll
    for (int s = kSubs - 1; s >= 0; --s) {
      post[s * D + c] = sum;
      sum += total[s];
    }
  }

  // ---- the blocks below the diagonal, on the tensor cores ----
  unsigned char* rows_k = planes;                      // [2][16][PB] k_i decayed from the block's start
  unsigned char* rows_q = rows_k + 2 * kSub * PB;      // [2][16][PB]
  unsigned char* columns = rows_q + 2 * kSub * PB;     // [2][48][PB] k_j decayed to the block's start
  constexpr int kColumnRows = (kSubs - 1) * kSub;
  for (int block = 1; block < kSubs; ++block) {
    for (int item = threadIdx.x; item < kSub * D / 4; item += kIntraThreads) {
      const int i = item / (D / 4), c = item % (D / 4) * 4, at = (block * kSub + i) * PD + c;
      const float4 f = exp2_4(*reinterpret_cast<const float4*>(xs + at));
      uint2 high, low;
      split4(mul4(*reinterpret_cast<const float4*>(ks + at), f), high, low);
      *reinterpret_cast<uint2*>(rows_k + i * PB + c * 2) = high;
      *reinterpret_cast<uint2*>(rows_k + (kSub + i) * PB + c * 2) = low;
      split4(mul4(*reinterpret_cast<const float4*>(qs + at), f), high, low);
      *reinterpret_cast<uint2*>(rows_q + i * PB + c * 2) = high;
      *reinterpret_cast<uint2*>(rows_q + (kSub + i) * PB + c * 2) = low;
    }
    for (int item = threadIdx.x; item < block * kSub * D / 4; item += kIntraThreads) {
      const int j = item / (D / 4), c = item % (D / 4) * 4, at = j * PD + c;
      float4 e = *reinterpret_cast<const float4*>(gs + at);
      for (int s = j / kSub + 1; s < block; ++s)
        e = add4(e, *reinterpret_cast<const float4*>(xs + (s * kSub + kSub - 1) * PD + c));
      uint2 high, low;
      split4(mul4(*reinterpret_cast<const float4*>(ks + at), exp2_4(e)), high, low);
      *reinterpret_cast<uint2*>(columns + j * PB + c * 2) = high;
      *reinterpret_cast<uint2*>(columns + (kColumnRows + j) * PB + c * 2) = low;
    }
    __syncthreads();
    const int tiles = block * 2;  // n8 tiles of a matrix
    for (int tile = warp; tile < 2 * tiles; tile += kIntraThreads / 32) {
      const bool is_q = tile < tiles;
      const int n0 = (is_q ? tile : tile - tiles) * 8;
      const uint32_t a_base = smem_u32(is_q ? rows_q : rows_k) + (lane & 15) * PB + (lane >> 4) * 16;
      const uint32_t b_base = smem_u32(columns) + (n0 + (lane & 7)) * PB + ((lane >> 3) & 1) * 16 + (lane >> 4) * kColumnRows * PB;
      float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f}, cross[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
      for (int step = 0; step < D / 16; ++step) {
        uint32_t ah[4], al[4], b[4];  // b: high (two registers), low
        ldmatrix_x4(ah, a_base + step * 32);
        ldmatrix_x4(al, a_base + kSub * PB + step * 32);
        ldmatrix_x4(b, b_base + step * 32);
        mma_bf16_16816(acc, ah, b[0], b[1]);
        mma_bf16_16816(cross, ah, b[2], b[3]);
        mma_bf16_16816(cross, al, b[0], b[1]);
      }
      float* matrix = is_q ? mixed : lower;
      const int r0 = block * kSub + (lane >> 2), c0 = n0 + (lane & 3) * 2;
      const float s0 = is_q ? 1.0f : betas[r0], s1 = is_q ? 1.0f : betas[r0 + 8];
      *reinterpret_cast<float2*>(matrix + r0 * PM + c0) = make_float2((acc[0] + cross[0]) * s0, (acc[1] + cross[1]) * s0);
      *reinterpret_cast<float2*>(matrix + (r0 + 8) * PM + c0) = make_float2((acc[2] + cross[2]) * s1, (acc[3] + cross[3]) * s1);
    }
    __syncthreads();
  }

  // ---- decayed operands of the second kernel; planes of the solve ----
#pragma unroll
  for (int i = 0; i < kRounds; ++i) {
    const int item = threadIdx.x + i * kIntraThreads, t = item / (D / 4), c = item % (D / 4) * 4, at = t * PD + c;
    const float4 into = add4(*reinterpret_cast<const float4*>(xs + at), *reinterpret_cast<const float4*>(pre + t / kSub * D + c));
    const float4 rest = add4(*reinterpret_cast<const float4*>(gs + at), *reinterpret_cast<const float4*>(post + t / kSub * D + c));
    uint2 high, low;
    split4(mul4(*reinterpret_cast<const float4*>(qs + at), exp2_4(into)), high, low);
    reinterpret_cast<uint2*>(out + Layout::kQ)[item] = high;
    reinterpret_cast<uint2*>(out + Layout::kQ + Layout::kPlane)[item] = low;
    split4(mul4(*reinterpret_cast<const float4*>(ks + at), exp2_4(rest)), high, low);
    reinterpret_cast<uint2*>(out + Layout::kK)[item] = high;
    reinterpret_cast<uint2*>(out + Layout::kK + Layout::kPlane)[item] = low;
  }
  __nv_bfloat16* triangle = reinterpret_cast<__nv_bfloat16*>(planes);      // [2][64][kTriangle]: minus the lower blocks
  __nv_bfloat16* inverse = triangle + 2 * kChunk * kTriangle;             // [2][64][kInverse]: inverted diagonal blocks
  for (int item = threadIdx.x; item < kChunk * kChunk / 4; item += kIntraThreads) {
    const int i = item / (kChunk / 4), j = item % (kChunk / 4) * 4;
    uint2 high, low;
    split4(*reinterpret_cast<const float4*>(mixed + i * PM + j), high, low);
    reinterpret_cast<uint2*>(out + Layout::kA)[item] = high;
    reinterpret_cast<uint2*>(out + Layout::kA + Layout::kSquare)[item] = low;
    if (j / kSub < i / kSub) {
      const float4 v = *reinterpret_cast<const float4*>(lower + i * PM + j);
      split4(make_float4(-v.x, -v.y, -v.z, -v.w), high, low);
      *reinterpret_cast<uint2*>(triangle + i * kTriangle + j) = high;
      *reinterpret_cast<uint2*>(triangle + (kChunk + i) * kTriangle + j) = low;
    }
  }
  invert_diagonal_blocks(lower, PM, inverse);
  __syncthreads();

  __nv_bfloat16* staging = reinterpret_cast<__nv_bfloat16*>(qs);  // [2][64][D] planes of W
  solve_chunk<D>(p, triangle, inverse, betas, staging, out, row0, count, head, warp, lane,
                 [&](int i, int c) { return ks[i * PD + c] * exp2f(xs[i * PD + c] + pre[i / kSub * D + c]); });
}

// ---- across the chunks -------------------------------------------------------------------
template <int D, int VB, bool DELTA>
constexpr int inter_smem_bytes() {
  return (DELTA ? 6 : 4) * kChunk * (D + 8) * 2 + 2 * kChunk * (kChunk + 8) * 2 + 2 * D * (VB + 8) * 2 + 2 * kChunk * (VB + 8) * 2;
}

// Warps: H share the columns of a 16-row tile, 16 C each. First product: 4 H warps on W S, 4 H on Q S;
// second: D / 16 x H warps on K^T U (their tile of S stays in registers), the last 4 H on A U.
template <int VB>
constexpr int kInterThreads = VB <= 32 ? VB * 16 : VB * 8;
template <int D, int VB, bool DELTA>
__global__ void __launch_bounds__(kInterThreads<VB>, 1) chunk_inter_kernel(const ChunkParams p) {
  constexpr int kThreads = kInterThreads<VB>, C = VB * 16 / kThreads, H = VB / (16 * C), T = 2 * C;  // T: n8 tiles of a warp
  constexpr int PB = (D + 8) * 2, PA = (kChunk + 8) * 2, PV = (VB + 8) * 2;  // byte pitches
  constexpr int kStateTiles = D / 16;
  using Layout = ChunkLayout<D>;
  extern __shared__ __align__(128) unsigned char smem[];
  unsigned char* q_planes = smem;                            // [2][64][PB]
  unsigned char* k_planes = q_planes + 2 * kChunk * PB;
  unsigned char* a_planes = k_planes + 2 * kChunk * PB;      // [2][64][PA]
  unsigned char* s_planes = a_planes + 2 * kChunk * PA;      // [2][D][PV]
  unsigned char* u_planes = s_planes + 2 * D * PV;           // [2][64][PV]
  unsigned char* w_planes = u_planes + 2 * kChunk * PV;      // [2][64][PB], delta
  const int head = blockIdx.y, sequence = blockIdx.z, v0 = blockIdx.x * VB;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slot = p.batch.slots[sequence];
  const int64_t first = p.batch.starts[sequence], last = p.batch.starts[sequence + 1];
  if (slot < 0) return;
  const int64_t per = Layout::bytes(DELTA, p.vdim);
  const int chunks = static_cast<int>((last - first + kChunk - 1) / kChunk);
  const unsigned char* in = p.workspace + (static_cast<int64_t>(p.chunk_starts[sequence]) * p.heads + head) * per;
  const int64_t stride = per * p.heads;
  auto copy = [&](unsigned char* dst, const unsigned char* src, auto row_bytes_constant, int pitch) {
    constexpr int row_bytes = decltype(row_bytes_constant)::value, chunks16 = row_bytes / 16;
#pragma unroll
    for (int item = threadIdx.x; item < 2 * kChunk * chunks16; item += kThreads) {
      const int r = item / chunks16, c = item % chunks16;
      cp_async16(smem_u32(dst + r * pitch + c * 16), src + static_cast<int64_t>(item) * 16);
    }
  };
  auto load_first = [&](int chunk) {  // operands of the products with S
    copy(q_planes, in + chunk * stride + Layout::kQ, IntConstant<D * 2>{}, PB);
    if (DELTA) copy(w_planes, in + chunk * stride + Layout::kW, IntConstant<D * 2>{}, PB);
    cp_async_commit();
  };
  auto load_second = [&](int chunk) {  // operands of the products with U
    copy(k_planes, in + chunk * stride + Layout::kK, IntConstant<D * 2>{}, PB);
    copy(a_planes, in + chunk * stride + Layout::kA, IntConstant<kChunk * 2>{}, PA);
    cp_async_commit();
  };
  load_first(0);
  load_second(0);

  const int half = warp % H;                          // which 16 C columns of this CTA's VB
  const int column = half * 16 * C + (lane & 3) * 2;  // this lane's first column of n8 tile 0
  const bool reads_out = warp >= 4 * H;         // Q S and A U; else W S and U
  const int tile = warp / H % 4, t_row = tile * 16 + (lane >> 2);
  const bool owns_state = warp / H < kStateTiles;
  const int s_row = warp / H * 16 + (lane >> 2);
  float* state = p.state + (static_cast<int64_t>(slot) * p.heads + head) * p.dim * p.state_row;
  const bool fresh = p.batch.bases[sequence] == 0;
  auto store_planes = [&](unsigned char* planes_at, int rows, int row, const float (*v)[4]) {
#pragma unroll
    for (int t = 0; t < T; ++t)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint32_t high, low;
        split_bf16x2(v[t][e * 2], v[t][e * 2 + 1], high, low);
        *reinterpret_cast<uint32_t*>(planes_at + (row + e * 8) * PV + (column + t * 8) * 2) = high;
        *reinterpret_cast<uint32_t*>(planes_at + (rows + row + e * 8) * PV + (column + t * 8) * 2) = low;
      }
  };
  float s[T][4] = {};
  if (owns_state) {
#pragma unroll
    for (int t = 0; t < T; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = s_row + (e >> 1) * 8, c = v0 + column + t * 8 + (e & 1);
        s[t][e] = !fresh && r < p.dim && c < p.vdim ? state[static_cast<int64_t>(r) * p.state_row + c] : 0.0f;
      }
    store_planes(s_planes, D, s_row, s);
  }
  const int v_row = (p.vdim + 31) / 32 * 32;
  float u0[T][4] = {}, end0 = 0.0f, end1 = 0.0f;  // fetched a chunk ahead
  auto fetch = [&](int chunk) {
    const int64_t row0 = first + static_cast<int64_t>(chunk) * kChunk;
    if (!reads_out) {
#pragma unroll
      for (int t = 0; t < T; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = t_row + (e >> 1) * 8, c = v0 + column + t * 8 + (e & 1);
          if (DELTA) u0[t][e] = c < v_row ? reinterpret_cast<const float*>(in + chunk * stride + Layout::kU)[r * v_row + c] : 0.0f;
          else u0[t][e] = row0 + r < last && c < p.vdim ? p.v[((row0 + r) * p.heads + head) * p.vdim + c] : 0.0f;
        }
    }
    if (owns_state) {
      const float* end = reinterpret_cast<const float*>(in + chunk * stride + Layout::kEnd);
      end0 = end[s_row];
      end1 = end[s_row + 8];
    }
  };
  fetch(0);
  cp_async_wait<1>();
  __syncthreads();

  // acc += A B: A given by its lanes' addresses (planes `a_low` bytes apart, `a_step` bytes a k16 step;
  // transposed when it lies [k][m]), B [k][VB] planes
  const uint32_t b_lane = (lane & 15) * PV + (lane >> 4) * 16 + half * 32 * C;
  auto product = [&](float (*acc)[4], auto transposed, uint32_t a, int a_low, int a_step, uint32_t b, int b_low,
                     auto steps) {
    float cross[T][4] = {};
#pragma unroll
    for (int step = 0; step < decltype(steps)::value; ++step) {
      uint32_t ah[4], al[4];
      if (decltype(transposed)::value != 0) {
        ldmatrix_x4_trans(ah, a + step * a_step);
        ldmatrix_x4_trans(al, a + a_low + step * a_step);
      } else {
        ldmatrix_x4(ah, a + step * a_step);
        ldmatrix_x4(al, a + a_low + step * a_step);
      }
#pragma unroll
      for (int c = 0; c < C; ++c) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bh, b + step * 16 * PV + c * 32);
        ldmatrix_x4_trans(bl, b + b_low + step * 16 * PV + c * 32);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma_bf16_16816(acc[c * 2 + t], ah, bh[t * 2], bh[t * 2 + 1]);
          mma_bf16_16816(cross[c * 2 + t], ah, bl[t * 2], bl[t * 2 + 1]);
          mma_bf16_16816(cross[c * 2 + t], al, bh[t * 2], bh[t * 2 + 1]);
        }
      }
    }
#pragma unroll
    for (int t = 0; t < T; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[t][e] += cross[t][e];
  };
  const uint32_t row_lane = (tile * 16 + (lane & 15)) * PB + (lane >> 4) * 16;
  const uint32_t s_base = smem_u32(s_planes) + b_lane, u_base = smem_u32(u_planes) + b_lane;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const int64_t row0 = first + static_cast<int64_t>(chunk) * kChunk;
    float acc[T][4] = {};
    if (reads_out) {
      product(acc, IntConstant<0>{}, smem_u32(q_planes) + row_lane, kChunk * PB, 32, s_base, D * PV, IntConstant<D / 16>{});
    } else {
      if (DELTA)
        product(acc, IntConstant<0>{}, smem_u32(w_planes) + row_lane, kChunk * PB, 32, s_base, D * PV, IntConstant<D / 16>{});
#pragma unroll
      for (int t = 0; t < T; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[t][e] = u0[t][e] - acc[t][e];
      store_planes(u_planes, kChunk, t_row, acc);
    }
    const float e0 = end0, e1 = end1;
    cp_async_wait<0>();
    __syncthreads();  // U is written, the second operands have landed, the first are free
    if (chunk + 1 < chunks) {
      load_first(chunk + 1);
      fetch(chunk + 1);
    }
    if (owns_state) {
#pragma unroll
      for (int t = 0; t < T; ++t) {
        s[t][0] *= e0; s[t][1] *= e0;
        s[t][2] *= e1; s[t][3] *= e1;
      }
      // the planes hold K [token][channel], so A = K^T is read transposed
      product(s, IntConstant<1>{}, smem_u32(k_planes) + ((lane & 7) + ((lane >> 4) << 3)) * PB + warp / H * 32 + ((lane >> 3) & 1) * 16,
              kChunk * PB, 16 * PB, u_base, kChunk * PV, IntConstant<kChunk / 16>{});
      store_planes(s_planes, D, s_row, s);
    }
    if (reads_out) {
      product(acc, IntConstant<0>{}, smem_u32(a_planes) + (tile * 16 + (lane & 15)) * PA + (lane >> 4) * 16, kChunk * PA, 32,
              u_base, kChunk * PV, IntConstant<kChunk / 16>{});
#pragma unroll
      for (int t = 0; t < T; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int64_t row = row0 + t_row + (e >> 1) * 8;
          const int c = v0 + column + t * 8 + (e & 1);
          if (row < last && c < p.vdim) p.output[(row * p.heads + head) * p.vdim + c] = acc[t][e];
        }
    }
    cp_async_wait<0>();
    __syncthreads();  // S is written, the first operands have landed, the second are free
    if (chunk + 1 < chunks) load_second(chunk + 1);
  }
  if (owns_state) {
#pragma unroll
    for (int t = 0; t < T; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = s_row + (e >> 1) * 8, c = v0 + column + t * 8 + (e & 1);
        if (r < p.dim && c < p.vdim) state[static_cast<int64_t>(r) * p.state_row + c] = s[t][e];
      }
  }
}

template <int D, bool DELTA>
int launch_chunked(const ChunkParams& p, int64_t chunks, bool head_decay, cudaStream_t stream) {
  auto intra = !DELTA ? chunk_intra_retention_kernel<D> : head_decay ? chunk_intra_head_delta_kernel<D>
                                                                     : chunk_intra_delta_kernel<D>;
  static_assert(intra_smem_bytes<D>() <= 226 * 1024, "the chunk does not fit shared memory");
  const int intra_smem = !DELTA ? 4 * kChunk * (D + 8) * 2 : head_decay ? intra_head_delta_smem_bytes<D>()
                                                                        : intra_smem_bytes<D>();
  if (cudaFuncSetAttribute(intra, cudaFuncAttributeMaxDynamicSharedMemorySize, intra_smem) != cudaSuccess)
    return B200_ERR_LAUNCH;
  intra<<<dim3(static_cast<unsigned>(chunks), static_cast<unsigned>(p.heads)),
          DELTA && head_decay ? kHeadDeltaThreads : kIntraThreads, intra_smem, stream>>>(p);
  auto inter = [&](auto kernel, int vb, int smem) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return B200_ERR_LAUNCH;
    kernel<<<dim3(static_cast<unsigned>(ceil_div(p.vdim, vb)), static_cast<unsigned>(p.heads),
                  static_cast<unsigned>(p.sequences)), vb <= 32 ? vb * 16 : vb * 8, smem, stream>>>(p);
    return launch_status();
  };
  // One CTA per SM: narrow column slices while the wide ones would leave half the SMs without a CTA, wide ones
  // (1.5 times the work's time) where they save as much in waves.
  const int64_t units = static_cast<int64_t>(p.heads) * p.sequences;
  const int64_t waves32 = ceil_div(ceil_div(p.vdim, 32) * units, kNumSMs), waves64 = ceil_div(ceil_div(p.vdim, 64) * units, kNumSMs);
  if (p.vdim > 32 && waves64 * 3 < waves32 * 2 + 1 && waves32 > 1)
    return inter(chunk_inter_kernel<D, 64, DELTA>, 64, inter_smem_bytes<D, 64, DELTA>());
  if (ceil_div(p.vdim, 32) * units * 2 > kNumSMs)
    return inter(chunk_inter_kernel<D, 32, DELTA>, 32, inter_smem_bytes<D, 32, DELTA>());
  return inter(chunk_inter_kernel<D, 16, DELTA>, 16, inter_smem_bytes<D, 16, DELTA>());
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" int64_t b200_recurrence_chunked_workspace_bytes(int64_t chunks, int64_t heads, int64_t dim, int64_t vdim,
                                                           int delta) {
  if (chunks <= 0 || heads <= 0 || dim <= 0 || dim > 128 || vdim <= 0 || vdim > 1024) return 0;
  const int64_t per = dim <= 64 ? ChunkLayout<64>::bytes(delta != 0, static_cast<int>(vdim))
                                : ChunkLayout<128>::bytes(delta != 0, static_cast<int>(vdim));
  return per * chunks * heads;
}

extern "C" int b200_recurrence_chunked(const float* q, const float* k, const float* v, const float* beta,
                                       const float* decay, float* state, float* output, const int32_t* token_sequence,
                                       const int32_t* starts, const int32_t* slots, const int32_t* bases,
                                       const int32_t* chunk_starts, int64_t chunks, int64_t sequences, int64_t heads,
                                       int64_t kv_heads, int64_t dim, int64_t vdim, int64_t state_row, int64_t decay_dim,
                                       void* workspace, int64_t workspace_bytes, void* stream) {
  if (!q || !k || !v || !decay || !state || !output || !starts || !slots || !bases || !chunk_starts || chunks < 0 ||
      sequences < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || dim <= 0 || vdim <= 0 || state_row < vdim ||
      (decay_dim != 1 && decay_dim != dim))
    return B200_ERR_BAD_ARGUMENT;
  if (dim > 128 || vdim > 1024) return B200_ERR_UNSUPPORTED;
  if (chunks == 0 || sequences == 0) return B200_OK;
  if (sequences > 65535 || heads > 65535 || chunks > INT32_MAX) return B200_ERR_TOO_LARGE;
  if (!workspace || workspace_bytes < b200_recurrence_chunked_workspace_bytes(chunks, heads, dim, vdim, beta != nullptr))
    return B200_ERR_WORKSPACE;
  if (!aligned16(workspace)) return B200_ERR_ALIGNMENT;
  ChunkParams p{q, k, v, beta, decay, state, output, {token_sequence, starts, slots, bases}, chunk_starts,
                static_cast<int>(sequences), static_cast<int>(heads), static_cast<int>(kv_heads), static_cast<int>(dim),
                static_cast<int>(vdim), static_cast<int>(state_row), static_cast<unsigned char*>(workspace)};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool head_decay = decay_dim != dim || dim == 1;
  if (dim <= 64)
    return beta ? launch_chunked<64, true>(p, chunks, head_decay, s) : launch_chunked<64, false>(p, chunks, false, s);
  return beta ? launch_chunked<128, true>(p, chunks, head_decay, s) : launch_chunked<128, false>(p, chunks, false, s);
}
