// Device helpers shared by the latent-attention kernels.
#pragma once
#include <cuda_bf16.h>
#include <math.h>
#include "mla.h"
#include "ptx_sm100.cuh"

namespace saber {

__device__ __forceinline__ float mla_warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float mla_warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
__device__ __forceinline__ int mla_seq_of_row(const int32_t* cu, int nseq, int m) {
  for (int j = 0; j < nseq; ++j)
    if (m < cu[j + 1]) return m >= cu[j] ? j : -1;
  return -1;
}
__device__ __forceinline__ float mla_gate(const MlaParams& p, int m, int h, int v) {
  return p.x[static_cast<size_t>(m) * p.ldx + p.g_off + (p.gate_heads ? h : h * p.V + v)];
}
// first key that the query at a position sees: of its chunk of positions, among the last `window`, or all (0, 0)
__device__ __forceinline__ int first_key(int pos, int chunk, int window) {
  if (window > 0) return max(0, pos - window + 1);
  return chunk > 0 ? pos - pos % chunk : 0;
}
// physical page of the i-th page of sequence j (bounds-checked: an entry outside the pool is recorded and read as page 0)
template <typename Params>
__device__ __forceinline__ int page_at(const Params& p, int j, int i) {
  const int b = i < p.max_blocks ? p.block_table[static_cast<size_t>(j) * p.max_blocks + i] : -1;
  if (b >= 0 && b < p.n_blocks) return b;
  if (p.err) atomicCAS(p.err, 0u, static_cast<uint32_t>(kErrBadIndex));
  return 0;
}

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ float ex2(float x) {     // 2^x, relative error 2^-22; -inf gives 0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool live) {   // !live: zero fill
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16u : 0u) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

}  // namespace saber

// mla_mma.cu: the bf16 forms on the tensor cores
int saber_mla_decode_attn(const saber::MlaParams* p, cudaStream_t stream);
int saber_mla_expand_attn(const saber::MlaParams* p, cudaStream_t stream);
bool saber_mla_decode_ok(const saber::MlaParams* p);
