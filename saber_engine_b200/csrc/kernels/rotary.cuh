// Rotary positions on the first `dims` values of a head: pair i turns by position * freq[i].
//   halves       pair i is (x[i], x[i + dims / 2])
//   interleaved  pair i is (x[2 i], x[2 i + 1])
// The table of one position holds amp cos, then amp sin of its dims / 2 angles (fp32).
#pragma once
#include <cuda_runtime.h>

namespace saber {

__device__ __forceinline__ void rotary_table(float* t, const float* freq, int dims, float amp, int pos, int tid, int threads) {
  const int half = dims / 2;
  for (int f = tid; f < half; f += threads) {
    float sn, cs;
    sincosf(static_cast<float>(pos) * freq[f], &sn, &cs);
    t[f] = amp * cs;
    t[half + f] = amp * sn;
  }
}

// rotated value d of the head at x (halves layout); values from `dims` on pass
__device__ __forceinline__ float rotary_half(const float* x, int d, const float* t, int dims) {
  if (d >= dims) return x[d];
  const int half = dims / 2;
  return d < half ? x[d] * t[d] - x[d + half] * t[half + d] : x[d] * t[d - half] + x[d - half] * t[d];
}

// rotated value d of the `dims` values at x, either layout
__device__ __forceinline__ float rotary_value(const float* x, int d, const float* t, int dims, bool interleaved) {
  if (!interleaved) return rotary_half(x, d, t, dims);
  const int f = d >> 1, half = dims / 2;
  return (d & 1) == 0 ? x[d] * t[f] - x[d + 1] * t[half + f] : x[d] * t[f] + x[d - 1] * t[half + f];
}

}  // namespace saber
