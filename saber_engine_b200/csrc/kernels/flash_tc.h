// Causal attention of prompt portions on tcgen05 (flash_tc.cu), over keys and values stored as tiles: keys
// [k-block of 64][64 tokens][128 bytes], values transposed [VP][64 tokens], 16-byte pieces XOR (row & 7).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>
#include "operand.cuh"

namespace saber {

struct FlashParams {
  const void* q;              // bf16 [M][H][DK]
  const void* k;              // of page p and key / value head g: k + (p G + g) k_stride bytes
  const void* v;
  size_t k_stride, v_stride;
  const float* gate;          // [M][ldg] (column h V + v, or h where gate_heads) through a sigmoid onto the output, or null
  int ldg, gate_heads;
  const float* sink;          // [H]: exp(sink) joins the denominator, or null
  const int32_t* cu_rows;     // [nseq + 1]
  const int32_t* kv_len;      // [nseq]
  const int32_t* block_table; // [nseq][max_blocks]
  Operand out;
  int out_k0;
  int nseq, H, G, DK, V, VP, n_blocks, max_blocks, max_rows;
  int chunk;                  // > 0: a row sees the keys of its own chunk of positions only
  int window;                 // > 0: a row sees the last `window` keys only, its own among them
  float out_scale;
  float scale, softcap;       // softcap > 0: scores cap tanh(scale s / cap)
  float bound;                // no |q . k| is larger (0: not known)
  uint32_t* err;
};

}  // namespace saber

bool saber_flash_tc_ok(int page, int DK, int VP, float scale, float softcap);
int saber_flash_tc(const saber::FlashParams* p, cudaStream_t stream);
