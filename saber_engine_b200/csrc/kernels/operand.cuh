// Token operand of the next linear, written by whichever kernel produces its values.
//   fmt 0  bf16, the GEMM's tile order: [k-block of 64][M_pad][128 bytes], 16-byte chunks XOR (m & 7)
//   fmt 1  fp32 rows [M_pad][ld]
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

namespace saber {

struct Operand {
  void* p;
  int M_pad, ld, fmt;
};

__device__ __forceinline__ size_t operand_chunk(const Operand& o, int m, int k) {   // byte offset of the 8-value chunk of k
  return (static_cast<size_t>(k >> 6) * o.M_pad + m) * 128 + (((((k & 63) >> 3) ^ m) & 7) << 4);
}

__device__ __forceinline__ void operand_store1(const Operand& o, int m, int k, float v) {
  if (o.fmt == 0)
    *reinterpret_cast<__nv_bfloat16*>(static_cast<uint8_t*>(o.p) + operand_chunk(o, m, k) + ((k & 7) << 1)) = __float2bfloat16(v);
  else
    static_cast<float*>(o.p)[static_cast<size_t>(m) * o.ld + k] = v;
}

// k a multiple of 4
__device__ __forceinline__ void operand_store4(const Operand& o, int m, int k, float4 v) {
  if (o.fmt == 0) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 w;
    w.x = *reinterpret_cast<const uint32_t*>(&a);
    w.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(static_cast<uint8_t*>(o.p) + operand_chunk(o, m, k) + ((k & 7) << 1)) = w;
  } else {
    *reinterpret_cast<float4*>(static_cast<float*>(o.p) + static_cast<size_t>(m) * o.ld + k) = v;
  }
}

// k a multiple of 8
__device__ __forceinline__ void operand_store8(const Operand& o, int m, int k, const float (&v)[8]) {
  if (o.fmt == 0) {
    uint4 w;
    uint32_t* u = reinterpret_cast<uint32_t*>(&w);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
      u[j] = *reinterpret_cast<const uint32_t*>(&b);
    }
    *reinterpret_cast<uint4*>(static_cast<uint8_t*>(o.p) + operand_chunk(o, m, k)) = w;
  } else {
    float4* d = reinterpret_cast<float4*>(static_cast<float*>(o.p) + static_cast<size_t>(m) * o.ld + k);
    d[0] = make_float4(v[0], v[1], v[2], v[3]);
    d[1] = make_float4(v[4], v[5], v[6], v[7]);
  }
}

__device__ __forceinline__ float operand_load1(const Operand& o, int m, int k) {
  if (o.fmt == 0)
    return __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(static_cast<const uint8_t*>(o.p) + operand_chunk(o, m, k) + ((k & 7) << 1)));
  return static_cast<const float*>(o.p)[static_cast<size_t>(m) * o.ld + k];
}

}  // namespace saber
