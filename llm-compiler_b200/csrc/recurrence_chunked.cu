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
// 16 bits of mantissa. Within 16 tokens the decayed products are built up token by token instead.
#include "common.cuh"
#include "hybrid.cuh"

namespace b200 {
namespace {

constexpr int kChunk = 64, kSub = 16, kSubs = kChunk / kSub;
constexpr int kIntraThreads = 256, kInterThreads = 256;

struct ChunkParams {
  const float *q, *k, *v;   // [rows, kv_heads, dim] x 2, [rows, heads, vdim]
  const float* beta;        // [rows, heads] (delta)
  const float* decay;       // log g [rows, heads, dim] (delta); decay [heads] (retention)
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
template <int D>
constexpr int intra_smem_bytes() {
  return 4 * kChunk * (D + 4) * 4 + 2 * kChunk * (kChunk + 4) * 4 + (2 * kSub + (kSubs - 1) * kSub) * 2 * (D + 8) * 2;
}

template <int D, bool DELTA>
__global__ void __launch_bounds__(kIntraThreads, 1) chunk_intra_kernel(const ChunkParams p) {
  constexpr int PD = D + 4, PM = kChunk + 4, PB = (D + 8) * 2;  // pitches: floats, floats, bytes
  using Layout = ChunkLayout<D>;
  extern __shared__ __align__(128) unsigned char smem[];
  float* ks = reinterpret_cast<float*>(smem);       // [64][PD]
  float* qs = ks + kChunk * PD;
  float* xs = qs + kChunk * PD;                     // log2 g, later its running sum within 16 tokens
  float* gs = xs + kChunk * PD;                     // g, later the sum of log2 g over the rest of the 16 tokens
  float* lower = gs + kChunk * PD;                  // [64][PM] beta_i k_i . (P_i / P_j) k_j, j < i
  float* mixed = lower + kChunk * PM;               // [64][PM] q_i . (P_i / P_j) k_j, j <= i
  unsigned char* planes = reinterpret_cast<unsigned char*>(mixed + kChunk * PM);
  __shared__ float betas[kChunk];
  __shared__ int sequence_slot;
  const int chunk = blockIdx.x, head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    int s = 0;
    while (s + 1 < p.sequences && p.chunk_starts[s + 1] <= chunk) ++s;
    sequence_slot = s;
  }
  __syncthreads();
  const int sequence = sequence_slot;
  const int64_t row0 = p.batch.starts[sequence] + static_cast<int64_t>(chunk - p.chunk_starts[sequence]) * kChunk;
  const int64_t left = p.batch.starts[sequence + 1] - row0;
  const int count = left < kChunk ? static_cast<int>(left) : kChunk;
  const int kv_head = head / (p.heads / p.kv_heads);
  unsigned char* out = p.workspace + (static_cast<int64_t>(chunk) * p.heads + head) * Layout::bytes(DELTA, p.vdim);
  const float head_decay = DELTA ? 0.0f : fmaxf(log2f(p.decay[head]), -126.0f);
  for (int item = threadIdx.x; item < kChunk * D; item += kIntraThreads) {
    const int t = item / D, c = item % D;
    const bool inside = t < count && c < p.dim;
    const int64_t source = inside ? ((row0 + t) * p.kv_heads + kv_head) * p.dim + c : 0;
    ks[t * PD + c] = inside ? p.k[source] : 0.0f;
    qs[t * PD + c] = inside ? p.q[source] : 0.0f;
    // (a token that keeps less than 2^-126 keeps nothing)
    float x = 0.0f;
    if (DELTA) x = inside ? fmaxf(p.decay[((row0 + t) * p.heads + head) * p.dim + c] * 1.4426950408889634f, -126.0f) : 0.0f;
    else x = t < count ? head_decay : 0.0f;
    xs[t * PD + c] = x;
    gs[t * PD + c] = exp2f(x);
  }
  if (threadIdx.x < kChunk)
    betas[threadIdx.x] = DELTA && threadIdx.x < count ? p.beta[(row0 + threadIdx.x) * p.heads + head] : 0.0f;
  for (int item = threadIdx.x; item < kChunk * PM; item += kIntraThreads) mixed[item] = 0.0f;
  __syncthreads();

  // ---- the 16 x 16 blocks on the diagonal: w = (P_i / P_j) k_j built up token by token ----
  {
    const int column = threadIdx.x >> 2, part = threadIdx.x & 3;  // four lanes a column, a quarter of the channels each
    const int block = column / kSub * kSub, j = column % kSub;
    float4 w[D / 16];
#pragma unroll
    for (int m = 0; m < D / 16; ++m) w[m] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    for (int i = 0; i < kSub; ++i) {
      const int at = (block + i) * PD + part * 4;
      float along_k = 0.0f, along_q = 0.0f;
#pragma unroll
      for (int m = 0; m < D / 16; ++m) {
        const float4 kk = *reinterpret_cast<const float4*>(ks + at + m * 16);
        const float4 qq = *reinterpret_cast<const float4*>(qs + at + m * 16);
        const float4 gg = *reinterpret_cast<const float4*>(gs + at + m * 16);
        if (i == j) {
          w[m] = kk;
        } else {
          w[m].x *= gg.x; w[m].y *= gg.y; w[m].z *= gg.z; w[m].w *= gg.w;
        }
        if (DELTA) along_k += kk.x * w[m].x + kk.y * w[m].y + kk.z * w[m].z + kk.w * w[m].w;
        along_q += qq.x * w[m].x + qq.y * w[m].y + qq.z * w[m].z + qq.w * w[m].w;
      }
      along_q += __shfl_xor_sync(0xffffffffu, along_q, 1);
      along_q += __shfl_xor_sync(0xffffffffu, along_q, 2);
      if (DELTA) {
        along_k += __shfl_xor_sync(0xffffffffu, along_k, 1);
        along_k += __shfl_xor_sync(0xffffffffu, along_k, 2);
      }
      if (part == 0) {
        if (DELTA) lower[(block + i) * PM + column] = i > j ? along_k * betas[block + i] : 0.0f;
        mixed[(block + i) * PM + column] = i >= j ? along_q : 0.0f;
      }
    }
  }
  __syncthreads();
  // ---- running sums of log2 g within 16 tokens, forwards (inclusive) and backwards (exclusive) ----
  for (int item = threadIdx.x; item < kSubs * D; item += kIntraThreads) {
    const int at = item / D * kSub * PD + item % D;
    float sum = 0.0f;
    for (int i = kSub - 1; i >= 0; --i) {
      gs[at + i * PD] = sum;
      sum += xs[at + i * PD];
    }
    sum = 0.0f;
    for (int i = 0; i < kSub; ++i) {
      sum += xs[at + i * PD];
      xs[at + i * PD] = sum;
    }
  }
  __syncthreads();
  auto total = [&](int sub, int c) { return xs[(sub * kSub + kSub - 1) * PD + c]; };
  auto before = [&](int t, int c) {  // log2 P_t
    float sum = xs[t * PD + c];
    for (int s = 0; s < t / kSub; ++s) sum += total(s, c);
    return sum;
  };
  auto after = [&](int t, int c) {  // log2 (P_last / P_t)
    float sum = gs[t * PD + c];
    for (int s = t / kSub + 1; s < kSubs; ++s) sum += total(s, c);
    return sum;
  };

  // ---- the blocks below the diagonal, on the tensor cores ----
  unsigned char* rows_k = planes;                      // [2][16][PB] k_i decayed from the block's start
  unsigned char* rows_q = rows_k + 2 * kSub * PB;      // [2][16][PB]
  unsigned char* columns = rows_q + 2 * kSub * PB;     // [2][48][PB] k_j decayed to the block's start
  constexpr int kColumnRows = (kSubs - 1) * kSub;
  for (int block = 1; block < kSubs; ++block) {
    for (int item = threadIdx.x; item < kSub * D / 2; item += kIntraThreads) {
      const int i = item / (D / 2), c = item % (D / 2) * 2, at = (block * kSub + i) * PD + c;
      const float f0 = exp2f(xs[at]), f1 = exp2f(xs[at + 1]);
      uint32_t high, low;
      if (DELTA) {
        split_bf16x2(ks[at] * f0, ks[at + 1] * f1, high, low);
        *reinterpret_cast<uint32_t*>(rows_k + i * PB + c * 2) = high;
        *reinterpret_cast<uint32_t*>(rows_k + (kSub + i) * PB + c * 2) = low;
      }
      split_bf16x2(qs[at] * f0, qs[at + 1] * f1, high, low);
      *reinterpret_cast<uint32_t*>(rows_q + i * PB + c * 2) = high;
      *reinterpret_cast<uint32_t*>(rows_q + (kSub + i) * PB + c * 2) = low;
    }
    for (int item = threadIdx.x; item < block * kSub * D / 2; item += kIntraThreads) {
      const int j = item / (D / 2), c = item % (D / 2) * 2, at = j * PD + c;
      float e0 = gs[at], e1 = gs[at + 1];
      for (int s = j / kSub + 1; s < block; ++s) {
        e0 += total(s, c);
        e1 += total(s, c + 1);
      }
      uint32_t high, low;
      split_bf16x2(ks[at] * exp2f(e0), ks[at + 1] * exp2f(e1), high, low);
      *reinterpret_cast<uint32_t*>(columns + j * PB + c * 2) = high;
      *reinterpret_cast<uint32_t*>(columns + (kColumnRows + j) * PB + c * 2) = low;
    }
    __syncthreads();
    const int tiles = block * 2;  // n8 tiles of a matrix
    for (int tile = warp; tile < (DELTA ? 2 : 1) * tiles; tile += kIntraThreads / 32) {
      const bool is_q = tile < tiles;
      const int n0 = (is_q ? tile : tile - tiles) * 8;
      const uint32_t a_base = smem_u32(is_q ? rows_q : rows_k) + (lane & 15) * PB + (lane >> 4) * 16;
      const uint32_t b_base = smem_u32(columns) + (n0 + (lane & 7)) * PB + ((lane >> 3) & 1) * 16 + (lane >> 4) * kColumnRows * PB;
      float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
      for (int step = 0; step < D / 16; ++step) {
        uint32_t ah[4], al[4], b[4];  // b: high (two registers), low
        ldmatrix_x4(ah, a_base + step * 32);
        ldmatrix_x4(al, a_base + kSub * PB + step * 32);
        ldmatrix_x4(b, b_base + step * 32);
        mma_bf16_16816(acc, ah, b[0], b[1]);
        mma_bf16_16816(acc, ah, b[2], b[3]);
        mma_bf16_16816(acc, al, b[0], b[1]);
      }
      float* matrix = is_q ? mixed : lower;
      const int r0 = block * kSub + (lane >> 2), c0 = n0 + (lane & 3) * 2;
      const float s0 = is_q ? 1.0f : betas[r0], s1 = is_q ? 1.0f : betas[r0 + 8];
      matrix[r0 * PM + c0] = acc[0] * s0;
      matrix[r0 * PM + c0 + 1] = acc[1] * s0;
      matrix[(r0 + 8) * PM + c0] = acc[2] * s1;
      matrix[(r0 + 8) * PM + c0 + 1] = acc[3] * s1;
    }
    __syncthreads();
  }

  // ---- decayed operands of the second kernel ----
  for (int item = threadIdx.x; item < kChunk * D / 2; item += kIntraThreads) {
    const int t = item / (D / 2), c = item % (D / 2) * 2, at = t * PD + c;
    uint32_t high, low;
    split_bf16x2(qs[at] * exp2f(before(t, c)), qs[at + 1] * exp2f(before(t, c + 1)), high, low);
    reinterpret_cast<uint32_t*>(out + Layout::kQ)[item] = high;
    reinterpret_cast<uint32_t*>(out + Layout::kQ + Layout::kPlane)[item] = low;
    split_bf16x2(ks[at] * exp2f(after(t, c)), ks[at + 1] * exp2f(after(t, c + 1)), high, low);
    reinterpret_cast<uint32_t*>(out + Layout::kK)[item] = high;
    reinterpret_cast<uint32_t*>(out + Layout::kK + Layout::kPlane)[item] = low;
  }
  for (int item = threadIdx.x; item < kChunk * kChunk / 2; item += kIntraThreads) {
    const int i = item / (kChunk / 2), j = item % (kChunk / 2) * 2;
    uint32_t high, low;
    split_bf16x2(mixed[i * PM + j], mixed[i * PM + j + 1], high, low);
    reinterpret_cast<uint32_t*>(out + Layout::kA)[item] = high;
    reinterpret_cast<uint32_t*>(out + Layout::kA + Layout::kSquare)[item] = low;
  }
  for (int c = threadIdx.x; c < D; c += kIntraThreads)
    reinterpret_cast<float*>(out + Layout::kEnd)[c] = exp2f(before(kChunk - 1, c));

  // ---- triangular solve, one column of (P k | v) a thread ----
  if (DELTA) {
    const int v_row = (p.vdim + 31) / 32 * 32;
    for (int column = threadIdx.x; column < D + v_row; column += kIntraThreads) {
      float x[kChunk];
      if (column < D) {
        float base = 0.0f;
#pragma unroll
        for (int i = 0; i < kChunk; ++i) {
          if (i > 0 && i % kSub == 0) base += total(i / kSub - 1, column);
          x[i] = betas[i] * ks[i * PD + column] * exp2f(base + xs[i * PD + column]);
        }
      } else {
        const int c = column - D;
#pragma unroll
        for (int i = 0; i < kChunk; ++i)
          x[i] = i < count && c < p.vdim ? betas[i] * p.v[((row0 + i) * p.heads + head) * p.vdim + c] : 0.0f;
      }
#pragma unroll
      for (int i = 1; i < kChunk; ++i) {
#pragma unroll
        for (int j = 0; j < i; j += 4) {
          const float4 l = *reinterpret_cast<const float4*>(lower + i * PM + j);
          x[i] = fmaf(-l.x, x[j], x[i]);
          if (j + 1 < i) x[i] = fmaf(-l.y, x[j + 1], x[i]);
          if (j + 2 < i) x[i] = fmaf(-l.z, x[j + 2], x[i]);
          if (j + 3 < i) x[i] = fmaf(-l.w, x[j + 3], x[i]);
        }
      }
      if (column < D) {
        __nv_bfloat16* high = reinterpret_cast<__nv_bfloat16*>(out + Layout::kW) + column;
        __nv_bfloat16* low = reinterpret_cast<__nv_bfloat16*>(out + Layout::kW + Layout::kPlane) + column;
#pragma unroll
        for (int i = 0; i < kChunk; ++i) {
          const __nv_bfloat16 h = __float2bfloat16_rn(x[i]);
          high[i * D] = h;
          low[i * D] = __float2bfloat16_rn(x[i] - __bfloat162float(h));
        }
      } else {
        float* u = reinterpret_cast<float*>(out + Layout::kU) + column - D;
#pragma unroll
        for (int i = 0; i < kChunk; ++i) u[i * v_row] = x[i];
      }
    }
  }
}

// ---- across the chunks -------------------------------------------------------------------
template <int D, int VB, bool DELTA>
constexpr int inter_smem_bytes() {
  return (DELTA ? 6 : 4) * kChunk * (D + 8) * 2 + 2 * kChunk * (kChunk + 8) * 2 + 2 * D * (VB + 8) * 2 + 2 * kChunk * (VB + 8) * 2;
}

template <int D, int VB, bool DELTA>
__global__ void __launch_bounds__(kInterThreads, 1) chunk_inter_kernel(const ChunkParams p) {
  constexpr int PB = (D + 8) * 2, PA = (kChunk + 8) * 2, PV = (VB + 8) * 2;  // byte pitches
  constexpr int NT = VB / 8;
  constexpr int kStateTiles = D / 16;  // warps that own a 16-row tile of S
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
  auto copy = [&](unsigned char* dst, const unsigned char* src, int rows, int row_bytes, int pitch) {
    const int chunks16 = row_bytes / 16;
    for (int item = threadIdx.x; item < rows * chunks16; item += kInterThreads) {
      const int r = item / chunks16, c = item % chunks16;
      cp_async16(smem_u32(dst + r * pitch + c * 16), src + static_cast<int64_t>(r) * row_bytes + c * 16);
    }
  };
  auto load_first = [&](int chunk) {  // operands of the products with S
    copy(q_planes, in + chunk * stride + Layout::kQ, 2 * kChunk, D * 2, PB);
    if (DELTA) copy(w_planes, in + chunk * stride + Layout::kW, 2 * kChunk, D * 2, PB);
    cp_async_commit();
  };
  auto load_second = [&](int chunk) {  // operands of the products with U
    copy(k_planes, in + chunk * stride + Layout::kK, 2 * kChunk, D * 2, PB);
    copy(a_planes, in + chunk * stride + Layout::kA, 2 * kChunk, kChunk * 2, PA);
    cp_async_commit();
  };
  load_first(0);
  load_second(0);

  // S: warp w owns rows 16 w .. 16 w + 15 of this CTA's columns, as an accumulator fragment
  float s[NT][4];
  const int s_row = warp * 16 + (lane >> 2), s_column = v0 + (lane & 3) * 2;
  float* state = p.state + (static_cast<int64_t>(slot) * p.heads + head) * p.dim * p.state_row;
  const bool fresh = p.batch.bases[sequence] == 0;
  auto store_planes = [&](unsigned char* planes_at, int rows, int row, int column, float a, float b) {
    uint32_t high, low;
    split_bf16x2(a, b, high, low);
    *reinterpret_cast<uint32_t*>(planes_at + row * PV + column * 2) = high;
    *reinterpret_cast<uint32_t*>(planes_at + (rows + row) * PV + column * 2) = low;
  };
  if (warp < kStateTiles) {
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = s_row + (e >> 1) * 8, c = s_column + t * 8 + (e & 1);
        s[t][e] = !fresh && r < p.dim && c < p.vdim ? state[static_cast<int64_t>(r) * p.state_row + c] : 0.0f;
      }
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      store_planes(s_planes, D, s_row, (lane & 3) * 2 + t * 8, s[t][0], s[t][1]);
      store_planes(s_planes, D, s_row + 8, (lane & 3) * 2 + t * 8, s[t][2], s[t][3]);
    }
  }
  cp_async_wait<1>();
  __syncthreads();

  // acc += A B with A [16 rows][k] K-major planes, B [k][VB] planes (row-major in shared memory)
  auto product = [&](float (&acc)[NT][4], uint32_t a_high, int a_low_offset, uint32_t b_high, int b_low_offset,
                     int steps) {
    for (int step = 0; step < steps; ++step) {
      uint32_t ah[4], al[4];
      ldmatrix_x4(ah, a_high + step * 32);
      ldmatrix_x4(al, a_high + a_low_offset + step * 32);
#pragma unroll
      for (int pair = 0; pair < NT / 2; ++pair) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bh, b_high + step * 16 * PV + pair * 32);
        ldmatrix_x4_trans(bl, b_high + b_low_offset + step * 16 * PV + pair * 32);
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          mma_bf16_16816(acc[pair * 2 + half], ah, bh[half * 2], bh[half * 2 + 1]);
          mma_bf16_16816(acc[pair * 2 + half], ah, bl[half * 2], bl[half * 2 + 1]);
          mma_bf16_16816(acc[pair * 2 + half], al, bh[half * 2], bh[half * 2 + 1]);
        }
      }
    }
  };
  const uint32_t b_lane = (lane & 15) * PV + (lane >> 4) * 16;
  const int v_row = (p.vdim + 31) / 32 * 32;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const int64_t row0 = first + static_cast<int64_t>(chunk) * kChunk;
    float acc[NT][4] = {};  // warps 0-3: W S, then U; warps 4-7: the read-out
    const int tile = warp & 3, t_row = tile * 16 + (lane >> 2);
    if (warp < 4) {
      float u0[NT][4];
#pragma unroll
      for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = t_row + (e >> 1) * 8, c = s_column + t * 8 + (e & 1);
          if (DELTA) u0[t][e] = c < v_row ? reinterpret_cast<const float*>(in + chunk * stride + Layout::kU)[r * v_row + c] : 0.0f;
          else u0[t][e] = row0 + r < last && c < p.vdim ? p.v[((row0 + r) * p.heads + head) * p.vdim + c] : 0.0f;
        }
      if (DELTA)
        product(acc, smem_u32(w_planes) + (tile * 16 + (lane & 15)) * PB + (lane >> 4) * 16, kChunk * PB,
                smem_u32(s_planes) + b_lane, D * PV, D / 16);
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        store_planes(u_planes, kChunk, t_row, (lane & 3) * 2 + t * 8, u0[t][0] - acc[t][0], u0[t][1] - acc[t][1]);
        store_planes(u_planes, kChunk, t_row + 8, (lane & 3) * 2 + t * 8, u0[t][2] - acc[t][2], u0[t][3] - acc[t][3]);
      }
    } else {
      product(acc, smem_u32(q_planes) + (tile * 16 + (lane & 15)) * PB + (lane >> 4) * 16, kChunk * PB,
              smem_u32(s_planes) + b_lane, D * PV, D / 16);
    }
    cp_async_wait<0>();
    __syncthreads();  // U is written, the second operands have landed, the first are free
    if (chunk + 1 < chunks) load_first(chunk + 1);
    if (warp < kStateTiles) {
      const float* end = reinterpret_cast<const float*>(in + chunk * stride + Layout::kEnd);
      const float e0 = end[s_row], e1 = end[s_row + 8];
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        s[t][0] *= e0; s[t][1] *= e0;
        s[t][2] *= e1; s[t][3] *= e1;
      }
      // S += K^T U: the planes hold K [token][channel], so A is read transposed
      const uint32_t a_base = smem_u32(k_planes) + ((lane & 7) + ((lane >> 4) << 3)) * PB + warp * 32 + ((lane >> 3) & 1) * 16;
#pragma unroll
      for (int step = 0; step < kChunk / 16; ++step) {
        uint32_t ah[4], al[4];
        ldmatrix_x4_trans(ah, a_base + step * 16 * PB);
        ldmatrix_x4_trans(al, a_base + kChunk * PB + step * 16 * PB);
#pragma unroll
        for (int pair = 0; pair < NT / 2; ++pair) {
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(bh, smem_u32(u_planes) + b_lane + step * 16 * PV + pair * 32);
          ldmatrix_x4_trans(bl, smem_u32(u_planes) + b_lane + kChunk * PV + step * 16 * PV + pair * 32);
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            mma_bf16_16816(s[pair * 2 + half], ah, bh[half * 2], bh[half * 2 + 1]);
            mma_bf16_16816(s[pair * 2 + half], ah, bl[half * 2], bl[half * 2 + 1]);
            mma_bf16_16816(s[pair * 2 + half], al, bh[half * 2], bh[half * 2 + 1]);
          }
        }
      }
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        store_planes(s_planes, D, s_row, (lane & 3) * 2 + t * 8, s[t][0], s[t][1]);
        store_planes(s_planes, D, s_row + 8, (lane & 3) * 2 + t * 8, s[t][2], s[t][3]);
      }
    }
    if (warp >= 4) {
      product(acc, smem_u32(a_planes) + (tile * 16 + (lane & 15)) * PA + (lane >> 4) * 16, kChunk * PA,
              smem_u32(u_planes) + b_lane, kChunk * PV, kChunk / 16);
#pragma unroll
      for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int64_t row = row0 + t_row + (e >> 1) * 8;
          const int c = s_column + t * 8 + (e & 1);
          if (row < last && c < p.vdim) p.output[(row * p.heads + head) * p.vdim + c] = acc[t][e];
        }
    }
    cp_async_wait<0>();
    __syncthreads();  // S is written, the first operands have landed, the second are free
    if (chunk + 1 < chunks) load_second(chunk + 1);
  }
  if (warp < kStateTiles) {
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = s_row + (e >> 1) * 8, c = s_column + t * 8 + (e & 1);
        if (r < p.dim && c < p.vdim) state[static_cast<int64_t>(r) * p.state_row + c] = s[t][e];
      }
  }
}

template <int D, bool DELTA>
int launch_chunked(const ChunkParams& p, int64_t chunks, cudaStream_t stream) {
  auto intra = chunk_intra_kernel<D, DELTA>;
  constexpr int intra_smem = intra_smem_bytes<D>();
  static_assert(intra_smem <= 226 * 1024, "the chunk does not fit shared memory");
  if (cudaFuncSetAttribute(intra, cudaFuncAttributeMaxDynamicSharedMemorySize, intra_smem) != cudaSuccess)
    return B200_ERR_LAUNCH;
  intra<<<dim3(static_cast<unsigned>(chunks), static_cast<unsigned>(p.heads)), kIntraThreads, intra_smem, stream>>>(p);
  auto inter = [&](auto kernel, int vb, int smem) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return B200_ERR_LAUNCH;
    kernel<<<dim3(static_cast<unsigned>(ceil_div(p.vdim, vb)), static_cast<unsigned>(p.heads),
                  static_cast<unsigned>(p.sequences)), kInterThreads, smem, stream>>>(p);
    return launch_status();
  };
  // narrow column slices while the wide ones would leave half the SMs without a CTA
  if (ceil_div(p.vdim, 32) * p.heads * p.sequences * 2 > kNumSMs)
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
                                       int64_t kv_heads, int64_t dim, int64_t vdim, int64_t state_row,
                                       void* workspace, int64_t workspace_bytes, void* stream) {
  if (!q || !k || !v || !decay || !state || !output || !starts || !slots || !bases || !chunk_starts || chunks < 0 ||
      sequences < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || dim <= 0 || vdim <= 0 || state_row < vdim)
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
  if (dim <= 64) return beta ? launch_chunked<64, true>(p, chunks, s) : launch_chunked<64, false>(p, chunks, s);
  return beta ? launch_chunked<128, true>(p, chunks, s) : launch_chunked<128, false>(p, chunks, s);
}
