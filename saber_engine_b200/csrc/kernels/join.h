// Launch interface of the row kernel between sublayers whose results are normed before they join the residual stream, and of
// the blend of neighbouring tokens ahead of a mixer (join.cu).  Plain C types only.
//
//   z = y + sum_k route_w[m][k] routed[slot_of[m][k]]      the sublayer's result: product rows, rows of routed experts, or both
//   x <- x + mult post_w z / rms(z) + step                 (fp32 stream; without a sublayer x + step, x from the embedding table)
//   h = norm_w x / rms(x)
//   op = h + shift (h' - h)                                h': the token before in its sequence (zeros ahead of the first)
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>
#include "operand.cuh"

namespace saber {

struct JoinParams {
  const float* y;             // [M][ldy] or null
  const void* routed;         // [rows][ldr], bf16 (routed_f32: fp32), or null
  const int32_t* slot_of;     // [M][routes], -1: none
  const float* route_w;
  const float* post_w;        // weights are padded with zeros to a multiple of 8
  const float* step;          // or null
  const void* table;          // bf16 or fp32 [vocab][width]: rows ids[m] times embed_scale instead of x, or null
  const int32_t* ids;
  const float* x;             // [M][ldx]
  float* x_out;               // [M][ldx]; x itself only without a blend
  const float* norm_w;
  Operand op;
  const float* shift;         // null: no blend
  float* state;               // [n_slots][width]: h of the sequence's last token
  const int32_t* cu_rows;     // [nseq + 1]
  const int32_t* slots;       // [nseq], < 0: padding sequence
  const int32_t* pos;         // [M]
  int M, width, ldx, ldy, ldr, routes, routed_f32, table_f32, vocab, nseq, n_slots;
  int rows;                   // rows of a CTA: 1, 2 or 4
  float mult, embed_scale, eps;
  uint32_t* err;
};

}  // namespace saber

extern "C" int saber_join_launch(const saber::JoinParams* p, cudaStream_t stream);
