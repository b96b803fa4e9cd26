// Launch interface of decayed outer products (ssd.cu, ssd_chunk.cu): linear attention and state-space mixers whose
// fp32 state S (N x V per head) obeys  S <- a S + k (w v)^T,  o = S^T q + skip v.  Plain C types only.
//
// q, k and v are silu of the projection, or of a causal convolution (with bias) over it; heads h .. share the
// key head h / (H / HK).  Decay and weight of a token:
//   constant   a = decay[h], w = 1                             (dt_off < 0)
//   selective  w = softplus(dt + dt_bias), a = exp(-exp(A_log) w)
// Read-out: the H V values in `groups` equal parts, each divided by its own root mean square, times norm_w, with
//   gate_first = 0   times sigmoid(gate) after the norm
//   gate_first = 1   times silu(gate) ahead of it
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>
#include "operand.cuh"

namespace saber {

struct SsdParams {
  const float* x;          // [M][ldx] projections of this step's rows
  int ldx, q_off, k_off, v_off, dt_off, g_off;
  const float* conv_w;     // [C][taps], C = 2 HK N + H V in q | k | v order, last column: the current token (taps = 0: none)
  const float* conv_b;     // [C]
  const float* decay;      // [H]
  const float* A_log;      // [H]
  const float* dt_bias;    // [H]
  const float* skip;       // [H] or null
  const float* norm_w;     // [H V]
  // state of a slot; the inputs of the convolution form a ring: the one of position p is row p % taps
  float* hist;             // [nslots][taps][C]
  float* state;            // [nslots][H][VP][DP] (pads stay zero)
  float* kq;               // scratch: the scan's records (scan_records.cuh)
  float* vb;
  float* o;                // scratch [M][H][VP]
  float* chunk;            // scratch of the chunk form (null: the scan)
  uint32_t* counters;      // [nseq][groups], zero between launches
  const int32_t* cu_rows;  // [nseq + 1]
  const int32_t* slots;    // [nseq], < 0: padding sequence
  const int32_t* pos;      // [M]
  Operand out;
  int out_k0;
  int M, nseq, H, HK, N, DP, V, VP, taps, groups, gate_first, n_slots;
  float eps;
  uint32_t* err;
};

}  // namespace saber

// single_row: every sequence brings at most one row (one fused launch)
extern "C" int saber_ssd_launches(const saber::SsdParams* p, int single_row);
extern "C" int saber_ssd_launch(const saber::SsdParams* p, int single_row, cudaStream_t stream);
