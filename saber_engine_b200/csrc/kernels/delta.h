// Launch interface of the gated delta rule with free sizes (delta.cu).  Plain C types only.
//
// Per head, with key size D and value size V (state S is D x V, fp32):
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// q, k: short causal convolution + silu, unit vectors per head (q also times q_scale); v: convolution + silu;
// beta = sigmoid(b), g = exp(-exp(A_log) softplus(a + dt_bias)); the read-out is divided by its root mean
// square over V, times norm_w, times silu(gate).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>
#include "operand.cuh"

namespace saber {

struct DeltaParams {
  const float* x;          // [M][ldx] projections of this step's rows
  int ldx, q_off, k_off, v_off, b_off, a_off, g_off;
  const float* conv_w;     // [C][taps], C = 2 HK D + H V in q | k | v order, last column: the current token
  const float* A_log;      // [H]
  const float* dt_bias;    // [H]
  const float* norm_w;     // [V]
  // state of a slot.  The inputs of the convolution form a ring: the one of position p is row p % taps, so a
  // step only overwrites rows that no later token reads.
  float* hist;             // [nslots][taps][C]
  float* state;            // [nslots][H][VP][DP] (pads stay zero)
  float* kq;               // scratch [M / 4 + nseq][HK][8 DP + 16]: blocks of four tokens, see delta.cu
  float* vb;               // scratch [M / 4 + nseq][H][ceil(VP / 16)][72]
  float* o;                // scratch [M][H][VP]
  const int32_t* cu_rows;  // [nseq + 1]
  const int32_t* slots;    // [nseq], < 0: padding sequence
  const int32_t* pos;      // [M] position of every row
  Operand out;
  int out_k0;
  int M, nseq, H, HK, D, DP, V, VP, taps, n_slots;
  float eps, unit_eps, q_scale;
  const float* skip;       // [H] or null: the scan without correction adds skip * v to the read-out
  uint32_t* err;
};

}  // namespace saber

// rows = 1: every sequence brings at most one row (one fused launch); else three launches
extern "C" int saber_delta_launches(int single_row);
extern "C" int saber_delta_launch(const saber::DeltaParams* p, int single_row, cudaStream_t stream);
// The scan by itself over records that another kernel has prepared, with the rule S <- g S + beta k v^T (no
// correction of v by what the state holds): decayed outer products (ssd.cu).
int saber_outer_scan_launch(const saber::DeltaParams* p, cudaStream_t stream);
