// Launch interface of the delta rule with a decay and a removal rate per key channel (cdelta.cu).  Plain C types only.
//
// Per head, with key size D and value size D (state S is D x D, fp32), from projections r, k, v, a, l of a token:
//   w = exp(-exp(-1/2) sigmoid(w0 + W2 tanh(l)))       decay of every key channel (l: `rank` values shared by the heads)
//   u = k / sqrt(|k|^2 + unit_eps)                     unit key
//   S <- diag(w) S - (sigmoid(a) u) (u^T S) + k v^T    both terms read the old state;   o = S^T r
// The read-out is divided by its root mean square over the head, times norm_w, times sigmoid(gate), times out_scale.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>
#include "operand.cuh"

namespace saber {

struct CdeltaParams {
  const float* x;             // [M][ldx] projections of this step's rows
  int ldx, r_off, k_off, v_off, a_off, l_off, g_off;
  const void* w2;             // [H D][rank, zeros up to a multiple of 16], bf16 (w2_f32: fp32)
  int w2_f32, rank;
  const float* w0;            // [H D]
  const float* norm_w;        // [H D]
  float* state;               // [n_slots][H][VP][DP] (pads stay zero)
  float* rec;                 // scratch [M / 4 + nseq][H][17 DP + 64]: blocks of four tokens, see cdelta.cu
  float* vb;                  // scratch [M / 4 + nseq][H][ceil(VP / 32)][128]
  float* o;                   // scratch [M][H][VP]
  const int32_t* cu_rows;     // [nseq + 1]
  const int32_t* slots;       // [nseq], < 0: padding sequence
  const int32_t* pos;         // [M]
  Operand out;
  int out_k0;
  int M, nseq, H, D, DP, VP, n_slots;
  float eps, unit_eps, out_scale;
  uint32_t* err;
};

}  // namespace saber

extern "C" int saber_cdelta_launches(int single_row);
extern "C" int saber_cdelta_launch(const saber::CdeltaParams* p, int single_row, cudaStream_t stream);
