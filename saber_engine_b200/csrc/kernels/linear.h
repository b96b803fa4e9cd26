// Launch interface of the linears whose residual stream is fp32 (linear.cu): a bf16 x bf16 tcgen05
// GEMM with the stream's epilogues, and the same linear in fp32 on the CUDA cores.  Plain C types only.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>
#include "operand.cuh"

namespace saber {

// What happens to acc[m][n] = sum_k a[m][k] w[n][k].  Two kinds:
//   project  the operand rows are norm_w * x without the division by the root mean square, so the
//            result is scaled by rsqrt(sum(ss[m]) * inv_width + eps) (ss: per-128-column sums of squares the
//            stream epilogue left; null: scale 1).  Features below act_tile0 * 256 are stored as fp32,
//            plus bias[n] (n < n_plain); those from there on are the feed-forward's and their activations go to
//            the operand `act`:
//              act_kind 0  a 256-feature tile holds 128 gate then 128 up features of a clamped gated unit,
//                          g = min(gate, limit), u = clamp(up, -limit, limit), y = g sigmoid(alpha g) (u + 1)
//              act_kind 1  y = max(up, 0)^2, 256 features a tile
//              act_kind 2  y = sigmoid(g) max(up, 0)^2, 248 features a tile and their gate's row g behind them
//              act_kind 3  y = gelu(up + act_bias) (by the error function), 256 features a tile
//              act_kind 4, 5  y = gelu(gate) up (by tanh), y = silu(gate) up, 128 gate then 128 up features a tile
//            The first lat_tiles tiles are a latent of lat_n values instead: the operand `lat` takes lat_w times the
//            value, lat_ss its sums of squares per 128 columns.  cap > 0: stored values become cap tanh(value / cap).
//   stream   x[m][n] = (add ? x[m][n] : 0) + bias[n] + acc, and the operand of the next linear:
//            norm_w[n] x[m][n] with its sums of squares (ss_out), or x itself (norm_w null).  norm_w2: a second
//            operand norm_w2[n] x[m][n] in op2.  y: rows of an expert product, acc[m] += sum_k route_w[m][k] y[slot_of[m][k]]
struct LinEpi {
  int stream;
  const float* ss;
  int ss_n;
  float inv_width, eps;
  float* out;
  int ldo, n_plain, act_tile0;
  Operand act;
  int act_k0, act_kind;
  float limit, alpha;
  float* x;
  int ldx, width, add;
  const float* bias;
  const float* norm_w;
  Operand op;
  int op_k0;
  float* ss_out;
  int ss_out_n;
  int lat_tiles, lat_n;
  Operand lat;
  const float* lat_w;
  float* lat_ss;
  int lat_ss_n;
  const float* act_bias;
  float cap;
  const float* norm_w2;
  Operand op2;
  const void* y;        // [rows][ldy], bf16 (y_f32: fp32)
  const int32_t* slot_of;
  const float* route_w;
  int routes, ldy, y_f32;
  int out_bf16;         // `out` is bf16 [M][ldo]
};

// group_tiles: a grouped product.  Row tile i is {expert, first row, rows}: rows of the (expert-major) output, each tile
// against the weight rows of its expert (group_w_stride bytes apart), at most nt mtiles rows (fp32: 64).  group_rows: the token of every
// output row, -1 between the experts' rows.  src_row: the same array where the operand's (and ss's) rows are tokens; null: they
// lie in output order.
struct LinParams {
  const void* w;        // bf16: [n_tile][k-block][32 KiB swizzled tile]; fp32: [N_pad][K]
  const void* a;        // bf16: operand tiles; fp32: rows [M_pad][K]
  const void* a2;       // operand of the weight tiles from a2_tile0 on (null: a)
  float* ws;            // split-K partials (bf16), the [M][N_pad] product (unfused forms)
  uint32_t* counters;   // one per output tile, zero between launches
  uint32_t* err;
  int M, M_pad, N_pad, K, nt, splits, fp32, fuse, mtiles;
  int a2_tile0;
  const int4* group_tiles;
  const int32_t* group_ntiles;
  const int32_t* group_rows;
  const int32_t* src_row;
  uint64_t group_w_stride;
  int group_max;        // tiles the table can hold
  LinEpi e;
};

// Rows of the stream from token ids: x = table[id] * scale, an optional second copy as the operand `x0`
// (columns from x0_k0), and the first layer's operand as in the stream epilogue.
struct StreamEmbedParams {
  const void* table;    // bf16 or fp32 [vocab][width]
  int table_f32, vocab;
  const int32_t* ids;
  int M, width;
  float scale;
  float* x;
  Operand x0;
  int x0_k0;            // < 0: none
  const float* norm_w;
  Operand op;
  int op_k0;
  float* ss_out;
  int ss_out_n;
  const float* norm_w2; // a second operand, columns from 0
  Operand op2;
};

// Stream rows `rows[i]` (null: row i), root-mean-square normed, as an operand.
struct StreamNormParams {
  const float* x;
  int ldx, width, n;
  const int32_t* rows;
  const float* w;
  float eps;
  Operand op;
};

}  // namespace saber

extern "C" int saber_linear_launches(const saber::LinParams* p);
extern "C" int saber_linear_launch(const saber::LinParams* p, cudaStream_t stream);
extern "C" int saber_stream_embed_launch(const saber::StreamEmbedParams* p, cudaStream_t stream);
extern "C" int saber_stream_norm_launch(const saber::StreamNormParams* p, cudaStream_t stream);
