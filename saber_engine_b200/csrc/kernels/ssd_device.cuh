// Device helpers of the decayed-outer-product kernels.
#pragma once
#include "ptx_sm100.cuh"
#include "scan_records.cuh"
#include "ssd.h"

namespace saber {

__device__ __forceinline__ int ssd_slot(const SsdParams& p, int j) {
  const int s = p.slots[j];
  if (s >= p.n_slots) {
    if (p.err) atomicCAS(p.err, 0u, static_cast<uint32_t>(kErrBadIndex));
    return -1;
  }
  return s;
}
__device__ __forceinline__ int ssd_channels(const SsdParams& p) { return 2 * p.HK * p.N + p.H * p.V; }
// column of channel c (q | k | v order) in a row of x
__device__ __forceinline__ int ssd_column(const SsdParams& p, int c) {
  const int kd = p.HK * p.N;
  return c < kd ? p.q_off + c : (c < 2 * kd ? p.k_off + c - kd : p.v_off + c - 2 * kd);
}
// decay a, its logarithm and the weight w of the token at row m
__device__ __forceinline__ void ssd_gates(const SsdParams& p, int m, int h, float& a, float& w, float& log_a) {
  if (p.dt_off < 0) {
    a = p.decay[h];
    w = 1.f;
    log_a = a > 0.f ? logf(a) : -1e4f;
    return;
  }
  w = softplus_f32(p.x[static_cast<size_t>(m) * p.ldx + p.dt_off + h] + p.dt_bias[h]);
  log_a = -expf(p.A_log[h]) * w;
  a = expf(log_a);
}
// silu of channel c's input at the ROWS rows from m on (m is row t of its sequence, at position pos); rows past
// `rows` (>= 1) give 0.  TAPS > 0: the number of taps when known at compile time; -1: no convolution; 0: p.taps of them.
template <int ROWS, int TAPS>
__device__ __forceinline__ void ssd_inputs(const SsdParams& p, const float* hist, int c, int m, int t, int pos, int C, int rows, float (&y)[ROWS]) {
  const int col = ssd_column(p, c);
  if constexpr (TAPS < 0) {
#pragma unroll
    for (int r = 0; r < ROWS; ++r) y[r] = p.x[static_cast<size_t>(m + min(r, rows - 1)) * p.ldx + col];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) y[r] = r < rows ? silu_f32(y[r]) : 0.f;
    return;
  }
  float acc[ROWS];
  const float b = p.conv_b ? p.conv_b[c] : 0.f;
#pragma unroll
  for (int r = 0; r < ROWS; ++r) acc[r] = b;
  const float* cw = p.conv_w + static_cast<size_t>(c) * p.taps;
  if constexpr (TAPS > 0) {
    float x[TAPS + ROWS - 1], w[TAPS];
#pragma unroll
    for (int i = 0; i < TAPS; ++i) w[i] = cw[i];
#pragma unroll
    for (int i = 0; i < TAPS + ROWS - 1; ++i) {                     // input row m - (TAPS - 1) + i
      const int back = TAPS - 1 - i;
      x[i] = 0.f;
      if (-back < rows) {
        if (back <= t) x[i] = p.x[static_cast<size_t>(m - back) * p.ldx + col];
        else if (back <= pos) x[i] = hist[static_cast<size_t>((pos - back) % TAPS) * C + c];
      }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
#pragma unroll
      for (int i = 0; i < TAPS; ++i) acc[r] = fmaf(x[r + i], w[i], acc[r]);
  } else {
    for (int back = p.taps - 1; back > -ROWS; --back) {             // input row m - back feeds rows r >= -back
      if (-back >= rows) break;
      float x = 0.f;
      if (back <= t) x = p.x[static_cast<size_t>(m - back) * p.ldx + col];
      else if (back <= pos) x = hist[static_cast<size_t>((pos - back) % p.taps) * C + c];
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const int i = p.taps - 1 - (r + back);
        if (i >= 0 && i < p.taps) acc[r] = fmaf(x, cw[i], acc[r]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < ROWS; ++r) y[r] = r < rows ? silu_f32(acc[r]) : 0.f;
}

}  // namespace saber
