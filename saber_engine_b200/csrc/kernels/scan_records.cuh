// What the prompt scan of delta.cu reads, and the small device functions its record writers share.
#pragma once
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

namespace saber {

__device__ __forceinline__ float warp_sum_f(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// (approximate division: two units in the last place; a denominator above 2^126 gives 0)
__device__ __forceinline__ float silu_f32(float x) { return __fdividef(x, 1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid_f32(float x) { return __fdividef(1.f, 1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f32(float x) { return x > 0.f ? x + log1pf(expf(-x)) : log1pf(expf(x)); }

// sequence of a row (-1: a padding row)
__device__ __forceinline__ int seq_of_row(const int32_t* cu, int nseq, int m) {
  for (int j = 0; j < nseq; ++j)
    if (m < cu[j + 1]) return m >= cu[j] ? j : -1;
  return -1;
}

constexpr int kBlk = 4;                  // tokens per block
constexpr int kPairs = 16;               // dot products per block: k_j . k_i (j < i: 6), k_j . q_i (j <= i: 10)
__host__ __device__ constexpr int kk_at(int i, int j) { return i * (i - 1) / 2 + j; }
__host__ __device__ constexpr int kq_at(int i, int j) { return 6 + i * (i + 1) / 2 + j; }

// Blocks of sequence j occupy the slots from (first row / 4) + j on: disjoint for all sequences of a step.
__device__ __forceinline__ int block_slot(int r0, int j, int c) { return (r0 >> 2) + j + c; }

// Scratch records of a block, each contiguous (one bulk copy):
//   key head   k rows [4][DP] | q rows [4][DP] | 16 dot products
//   value head, per 16 columns   v [4][16] | beta [4] | g [4]
// Missing tokens of the last block are written as k = q = v = beta = 0, g = 1.
__host__ __device__ constexpr int kq_words(int DP) { return 2 * kBlk * DP + kPairs; }
constexpr int kCols = 16;                // value columns of a scan CTA
constexpr int kVWords = kBlk * kCols + 2 * kBlk;

}  // namespace saber
