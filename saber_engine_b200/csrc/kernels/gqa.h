// Launch interface of grouped-query attention over tiled pages (gqa.cu): H query heads share G key / value heads,
// fp32 scores.  Plain C types only.
//
//   q, k    optionally divided by their root mean square over D (qk_norm), then rotated (rot > 0: the first rot values, halves
//           layout)
//   taps    > 0: q, k and v first pass a causal convolution of their own over the tokens; q and k are then normed over all heads at once
//           (weights q_w, k_w), values per head (v_norm)
//   score   scale q . k, then cap tanh(score / cap) when softcap > 0
//   sink    exp(sink[h]) joins the denominator of head h
//   gate    the output times sigmoid of column g_off + h V + v of x
//   mask    keys j <= i; chunk > 0: of the same chunk of positions as i only, j >= i - i % chunk; window > 0: the last
//           `window` ones only, i itself among them
//
// A page holds, per key / value head, the keys and then the values of its 64 tokens.  bf16: in the order the
// tensor-core kernels multiply in place, keys [D / 64][64 tokens][128 bytes], values transposed [VP][64 tokens], both
// with 16-byte pieces XOR (row & 7).  fp32: keys [64][KP], values [64][VP].
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>
#include "operand.cuh"

namespace saber {

struct GqaParams {
  const float* x;             // [M][ldx] projections of this step's rows
  int ldx, q_off, k_off, v_off;   // k_off < 0: the cache is another layer's, nothing is appended
  int g_off;                      // < 0: no gate
  int rot;
  float rot_amp;
  const float* freq;          // [rot / 2]
  const float* sink;          // [H] or null
  void* cache;                // [n_blocks][G][64 (KP + VP)]
  void* q;                    // scratch [M][H][DK] bf16 (tcgen05 form)
  float* o_part;              // scratch [M][H][splits][VP]
  float* ml;                  // scratch [M][H][splits][2]
  uint32_t* counters;         // [M][G], zero between launches
  const int32_t* slot_map;    // [M] page * 64 + offset, -1: padding row
  const int32_t* pos;         // [M]
  const int32_t* cu_rows;     // [nseq + 1]
  const int32_t* kv_len;      // [nseq]
  const int32_t* block_table; // [nseq][max_blocks]
  Operand out;
  int out_k0;
  int M, nseq, H, G, D, DK, KP, V, VP, page, n_blocks, max_blocks, splits;
  int f32;                    // element type of the cache
  int form;                   // 0: a CTA per (row, head), any size; 1: mma.sync over split keys; 2: tcgen05
  int max_rows;               // rows one sequence may bring (1: the split form appends the row's key by itself)
  int qk_norm, chunk;
  float scale, softcap, eps;
  uint32_t* err;
  int window;
  float out_scale;            // factor of the output
  // convolution (taps > 0).  Inputs of a slot form a ring: the one of position p is row p % taps.
  int taps, v_norm, n_slots, ldc;
  const float* conv_w;        // [taps][C], C = H D + G D + G V in q | k | v order, last row: the current token
  const float* q_w;           // [H D]
  const float* k_w;           // [G D]
  float* hist;                // [n_slots][taps][C]
  const int32_t* slots;       // [nseq]
  float* cx;                  // scratch [M][ldc]: the convolved rows, q | k | v from multiples of 8 on
  float* row_ss;              // scratch [M][ceil(H D / 256) + ceil(G D / 256)]: sums of squares of 256 columns each, q's then k's
  // set at the launch
  const float* gate;          // column 0 of the gate in row 0
  int ld_gate;
  const float* raw;           // the rows ahead of the convolution
  int ld_raw, rq_off, rk_off, rv_off;
};

}  // namespace saber

extern "C" int saber_gqa_form(const saber::GqaParams* p);     // the best form for these sizes
extern "C" int saber_gqa_launches(const saber::GqaParams* p);
extern "C" int saber_gqa_launch(const saber::GqaParams* p, cudaStream_t stream);
