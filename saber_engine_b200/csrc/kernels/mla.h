// Launch interface of latent attention (mla.cu): per token one latent row c (kv_rank values, shared by
// every head) and one rotated key part are cached; a head's key is [W_uk c | rotated part], its value
// W_uv c.  Plain C types only.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>
#include "operand.cuh"

namespace saber {

struct MlaParams {
  const float* x;             // [M][ldx] projections of this step's rows
  int ldx, q_off, dkv_off, g_off;   // dkv_off < 0: the cache is another layer's, nothing is appended
  const float* q;             // [M][ldq] queries (column q_off on)
  int ldq;
  int gate_heads;             // 1: one gate per head (column g_off + h), 0: one per value (g_off + h V + v)
  int interleaved;            // layout of a rotated pair (rotary.cuh)
  float rot_amp;
  const float* dkv_norm;      // [C]
  const float* freq;          // [R / 2] rotary frequencies
  const void* w_uk;           // [H * D][CP] (pads zero)
  const void* w_uv;           // [H * V][CP]
  void* cache;                // [n_blocks][page][CP + RP]: latent, rotated key (pads zero)
  void* q_eff;                // scratch [M][H][max(CP, DP) + RP]
  float* o_part;              // scratch [M][H][splits][CP] (absorbed form)
  float* ml;                  // scratch [M][H][splits][2]
  // expanded form (prompt portions, bf16): keys and values of the pages this step sees, in physical page order
  void* k_exp;                // [n_blocks][H][page][DP + RP]; expand = 2: tiles [n_blocks][H][ceil((DP + RP) / 64)][page][64]
  void* v_exp;                // [n_blocks][H][page][VP]; expand = 2: transposed [n_blocks][H][VP][page]
  const int32_t* slot_map;    // [M] page * page_tokens + offset, -1: padding row
  const int32_t* pos;         // [M]
  const int32_t* cu_rows;     // [nseq + 1]
  const int32_t* kv_len;      // [nseq]
  const int32_t* block_table; // [nseq][max_blocks]
  Operand out;
  int out_k0;
  int M, nseq, H, D, R, V, C, CP, RP, DP, VP, page, n_blocks, max_blocks, splits;
  int f32;                    // element type of cache, weights and q_eff: fp32 or bf16
  int expand;                 // expanded form: 1 mma.sync, 2 tcgen05; 0: absorbed form
  int max_rows;               // rows one sequence may bring
  float scale, eps;
  uint32_t* err;
};

}  // namespace saber

extern "C" int saber_mla_expand_ok(const saber::MlaParams* p);
extern "C" int saber_mla_launches(const saber::MlaParams* p);
extern "C" int saber_mla_launch(const saber::MlaParams* p, cudaStream_t stream);
