// Gated delta rule with free head sizes, fp32 throughout.
//
// Prompt portions (ragged rows, any length): three launches.
//   prep   one CTA row by row: convolution, silu, unit norms, beta and decay
//   scan   the recurrence.  Columns of the state are independent, so a warp owns eight value columns
//          for the whole portion: eight lanes split the key dimension, four lane groups take two columns
//          each, the state stays in registers, and both products of a token (S^T k and S^T q; the
//          read-out after the write is g S^T q + u (k . q)) meet in one three-step shuffle reduction.
//          Eight tokens at a time are staged in shared memory by asynchronous copies, double buffered.
//   out    gated norm into the operand of the output linear; the convolution inputs go to the ring
// Decoding (one row per sequence): all of it in one launch, a CTA per (head, sequence).
#include "delta.h"
#include "launch.cuh"
#include "ptx_sm100.cuh"

namespace saber {

constexpr int kDeltaMaxPerLane = 16;     // head sizes up to 512

__device__ __forceinline__ float warp_sum_f(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float silu_f32(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid_f32(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f32(float x) { return x > 0.f ? x + log1pf(expf(-x)) : log1pf(expf(x)); }

// sequence of a row (-1: a padding row), and whether its slot may be used
__device__ __forceinline__ int seq_of_row(const int32_t* cu, int nseq, int m) {
  for (int j = 0; j < nseq; ++j)
    if (m < cu[j + 1]) return m >= cu[j] ? j : -1;
  return -1;
}
__device__ __forceinline__ int delta_slot(const DeltaParams& p, int j) {
  const int s = p.slots[j];
  if (s >= p.n_slots) {
    if (p.err) atomicCAS(p.err, 0u, static_cast<uint32_t>(kErrBadIndex));
    return -1;
  }
  return s;
}

// convolution + silu of channel c at row m (col: the channel's column in x); t = row inside its sequence
__device__ __forceinline__ float conv_silu(const DeltaParams& p, const float* hist, int c, int col, int m, int t, int pos, int C) {
  float acc = 0.f;
  for (int i = 0; i < p.taps; ++i) {
    const int back = p.taps - 1 - i;
    float x = 0.f;
    if (back <= t) x = p.x[static_cast<size_t>(m - back) * p.ldx + col];
    else if (back <= pos) x = hist[static_cast<size_t>((pos - back) % p.taps) * C + c];
    acc = fmaf(x, p.conv_w[static_cast<size_t>(c) * p.taps + i], acc);
  }
  return silu_f32(acc);
}

// grid (M, ceil(items / 8)); a warp per item: q heads, k heads, v heads, then one item for beta / decay
__global__ void __launch_bounds__(256) delta_prep_kernel(const __grid_constant__ DeltaParams p) {
  pdl_wait();
  const int m = blockIdx.x;
  const int lane = threadIdx.x & 31;
  const int item = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (item > 2 * p.HK + p.H) return;
  const int j = seq_of_row(p.cu_rows, p.nseq, m);
  if (j < 0) return;
  const int slot = delta_slot(p, j);
  if (slot < 0) return;
  const int t = m - p.cu_rows[j], pos = p.pos[m];
  const int C = 2 * p.HK * p.D + p.H * p.V;
  const float* hist = p.hist + static_cast<size_t>(slot) * p.taps * C;
  if (item < 2 * p.HK) {
    const bool isq = item < p.HK;
    const int h = isq ? item : item - p.HK;
    const int c0 = (isq ? 0 : p.HK * p.D) + h * p.D, col0 = (isq ? p.q_off : p.k_off) + h * p.D;
    float v[kDeltaMaxPerLane];
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < kDeltaMaxPerLane; ++i) {
      const int d = i * 32 + lane;
      v[i] = 0.f;
      if (d < p.D) v[i] = conv_silu(p, hist, c0 + d, col0 + d, m, t, pos, C);
      sq += v[i] * v[i];
    }
    const float r = 1.f / sqrtf(warp_sum_f(sq) + p.unit_eps) * (isq ? p.q_scale : 1.f);
    float* o = (isq ? p.qn : p.kn) + (static_cast<size_t>(m) * p.HK + h) * p.DP;
#pragma unroll
    for (int i = 0; i < kDeltaMaxPerLane; ++i)
      if (i * 32 + lane < p.DP) o[i * 32 + lane] = v[i] * r;
  } else if (item < 2 * p.HK + p.H) {
    const int h = item - 2 * p.HK;
    float* o = p.vv + (static_cast<size_t>(m) * p.H + h) * p.VP;
    for (int d = lane; d < p.VP; d += 32)
      o[d] = d < p.V ? conv_silu(p, hist, 2 * p.HK * p.D + h * p.V + d, p.v_off + h * p.V + d, m, t, pos, C) : 0.f;
  } else {
    const float* x = p.x + static_cast<size_t>(m) * p.ldx;
    for (int h = lane; h < p.H; h += 32) {
      float* o = p.bg + (static_cast<size_t>(m) * p.H + h) * 2;
      o[0] = sigmoid_f32(x[p.b_off + h]);
      o[1] = expf(-expf(p.A_log[h]) * softplus_f32(x[p.a_off + h] + p.dt_bias[h]));
    }
  }
}

// One token on the state columns of a lane (two of the warp's eight).
template <int NI>
__device__ __forceinline__ void delta_token(float (&S)[NI][4][2], const float* k, const float* q, int lg, float v0, float v1, float beta,
                                            float g, float& o0, float& o1) {
  float sk0 = 0.f, sk1 = 0.f, sq0 = 0.f, sq1 = 0.f, kq = 0.f;
  float4 kr[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    kr[i] = *reinterpret_cast<const float4*>(k + i * 32 + lg * 4);
    const float4 qr = *reinterpret_cast<const float4*>(q + i * 32 + lg * 4);
    const float ka[4] = {kr[i].x, kr[i].y, kr[i].z, kr[i].w};
    const float qa[4] = {qr.x, qr.y, qr.z, qr.w};
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      sk0 = fmaf(S[i][r][0], ka[r], sk0);
      sk1 = fmaf(S[i][r][1], ka[r], sk1);
      sq0 = fmaf(S[i][r][0], qa[r], sq0);
      sq1 = fmaf(S[i][r][1], qa[r], sq1);
      kq = fmaf(ka[r], qa[r], kq);
    }
  }
#pragma unroll
  for (int o = 1; o < 8; o <<= 1) {
    sk0 += __shfl_xor_sync(0xffffffffu, sk0, o);
    sk1 += __shfl_xor_sync(0xffffffffu, sk1, o);
    sq0 += __shfl_xor_sync(0xffffffffu, sq0, o);
    sq1 += __shfl_xor_sync(0xffffffffu, sq1, o);
    kq += __shfl_xor_sync(0xffffffffu, kq, o);
  }
  const float u0 = beta * (v0 - g * sk0), u1 = beta * (v1 - g * sk1);
  o0 = fmaf(u0, kq, g * sq0);
  o1 = fmaf(u1, kq, g * sq1);
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const float ka[4] = {kr[i].x, kr[i].y, kr[i].z, kr[i].w};
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      S[i][r][0] = fmaf(u0, ka[r], g * S[i][r][0]);
      S[i][r][1] = fmaf(u1, ka[r], g * S[i][r][1]);
    }
  }
}

template <int NI>
__device__ __forceinline__ void delta_state_io(float* st, float (&S)[NI][4][2], int DP, int lg, bool store) {
#pragma unroll
  for (int c = 0; c < 2; ++c)
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      float4* a = reinterpret_cast<float4*>(st + static_cast<size_t>(c) * DP + i * 32 + lg * 4);
      if (store) {
        *a = make_float4(S[i][0][c], S[i][1][c], S[i][2][c], S[i][3][c]);
      } else {
        const float4 f = *a;
        S[i][0][c] = f.x; S[i][1][c] = f.y; S[i][2][c] = f.z; S[i][3][c] = f.w;
      }
    }
}

constexpr int kScanRows = 8;

// grid (nseq, H, ceil(VP / 32)), 128 threads
template <int NI>
__global__ void __launch_bounds__(128) delta_scan_kernel(const __grid_constant__ DeltaParams p) {
  pdl_wait();
  extern __shared__ float4 sm4[];
  float* sm = reinterpret_cast<float*>(sm4);
  constexpr int DP = NI * 32;
  constexpr int kRow = 2 * DP + 32 + 4;            // k | q | 32 value columns | beta, g
  const int j = blockIdx.x, h = blockIdx.y;
  const int r0 = p.cu_rows[j], n = p.cu_rows[j + 1] - r0;
  if (n <= 0) return;
  const int slot = delta_slot(p, j);
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 7;
  const int vb = blockIdx.z * 32, nv = min(32, p.VP - vb);
  const int hk = h / (p.H / p.HK);
  const int cl = warp * 8 + (lane >> 3) * 2;       // column inside the CTA's 32
  const bool on = warp * 8 < nv;                   // VP is a multiple of 8
  float S[NI][4][2] = {};
  float* st = p.state + ((static_cast<size_t>(slot) * p.H + h) * p.VP + vb + cl) * DP;
  if (on) delta_state_io<NI>(st, S, DP, lg, false);

  auto fetch = [&](int c) {                        // rows [c * kScanRows, ...) into buffer c & 1
    float* b = sm + (c & 1) * kScanRows * kRow;
    const int rows = min(kScanRows, n - c * kScanRows);
    for (int i = threadIdx.x; i < rows * (kRow / 4); i += 128) {
      const int r = i / (kRow / 4), w = i - r * (kRow / 4);
      const size_t m = r0 + c * kScanRows + r;
      const float* src;
      if (w < DP / 4) src = p.kn + (m * p.HK + hk) * DP + w * 4;
      else if (w < DP / 2) src = p.qn + (m * p.HK + hk) * DP + (w - DP / 4) * 4;
      else if (w < DP / 2 + 8) {
        const int v = (w - DP / 2) * 4;
        if (v >= nv) continue;
        src = p.vv + (m * p.H + h) * p.VP + vb + v;
      } else {
        // beta, g: eight bytes
        const float* s2 = p.bg + (m * p.H + h) * 2;
        asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(smem_u32(b + r * kRow + w * 4)), "l"(s2) : "memory");
        continue;
      }
      asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"(smem_u32(b + r * kRow + w * 4)), "l"(src) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int chunks = (n + kScanRows - 1) / kScanRows;
  fetch(0);
  for (int c = 0; c < chunks; ++c) {
    if (c + 1 < chunks) {
      fetch(c + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    if (on) {
      const float* b = sm + (c & 1) * kScanRows * kRow;
      const int rows = min(kScanRows, n - c * kScanRows);
      for (int r = 0; r < rows; ++r, b += kRow) {
        const float2 v = *reinterpret_cast<const float2*>(b + 2 * DP + cl);
        const float2 bg = *reinterpret_cast<const float2*>(b + 2 * DP + 32);
        float o0, o1;
        delta_token<NI>(S, b, b + DP, lg, v.x, v.y, bg.x, bg.y, o0, o1);
        if (lg == 0)
          *reinterpret_cast<float2*>(p.o + (static_cast<size_t>(r0 + c * kScanRows + r) * p.H + h) * p.VP + vb + cl) = make_float2(o0, o1);
      }
    }
    __syncthreads();
  }
  if (on) delta_state_io<NI>(st, S, DP, lg, true);
}

// Gated norm of one head row (o: V values, shared or global memory) by a warp.
__device__ __forceinline__ void delta_gated_norm(const DeltaParams& p, const float* o, int m, int h, int lane) {
  float sq = 0.f;
  for (int v = lane; v < p.V; v += 32) sq += o[v] * o[v];
  const float r = 1.f / sqrtf(warp_sum_f(sq) / static_cast<float>(p.V) + p.eps);
  const float* g = p.x + static_cast<size_t>(m) * p.ldx + p.g_off + h * p.V;
  for (int v = lane; v < p.V; v += 32) operand_store1(p.out, m, p.out_k0 + h * p.V + v, o[v] * r * p.norm_w[v] * silu_f32(g[v]));
}

// grid (M + nseq, ceil(H / 8)): a warp per (row, head); the last nseq rows of the grid update the rings
__global__ void __launch_bounds__(256) delta_out_kernel(const __grid_constant__ DeltaParams p) {
  pdl_wait();
  const int lane = threadIdx.x & 31;
  if (static_cast<int>(blockIdx.x) < p.M) {
    const int m = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5);
    if (h >= p.H || seq_of_row(p.cu_rows, p.nseq, m) < 0) return;
    delta_gated_norm(p, p.o + (static_cast<size_t>(m) * p.H + h) * p.VP, m, h, lane);
    return;
  }
  const int j = blockIdx.x - p.M;
  const int r0 = p.cu_rows[j], n = p.cu_rows[j + 1] - r0;
  const int slot = n > 0 ? delta_slot(p, j) : -1;
  if (slot < 0) return;
  const int C = 2 * p.HK * p.D + p.H * p.V, kd = p.HK * p.D;
  float* hist = p.hist + static_cast<size_t>(slot) * p.taps * C;
  for (int c = blockIdx.y * 256 + threadIdx.x; c < C; c += gridDim.y * 256) {
    const int col = c < kd ? p.q_off + c : (c < 2 * kd ? p.k_off + c - kd : p.v_off + c - 2 * kd);
    for (int t = max(0, n - p.taps); t < n; ++t) {
      const int m = r0 + t;
      hist[static_cast<size_t>(p.pos[m] % p.taps) * C + c] = p.x[static_cast<size_t>(m) * p.ldx + col];
    }
  }
}

// One row per sequence: grid (H, nseq), 32 * min(8, VP / 8) threads.
template <int NI>
__global__ void __launch_bounds__(256) delta_step_kernel(const __grid_constant__ DeltaParams p) {
  pdl_wait();
  extern __shared__ float4 sm4[];
  constexpr int DP = NI * 32;
  float* ks = reinterpret_cast<float*>(sm4);       // DP
  float* qs = ks + DP;                             // DP
  float* vs = qs + DP;                             // VP
  float* os = vs + p.VP;                           // VP
  __shared__ float red[2][8], sum_s[2];
  const int h = blockIdx.x, j = blockIdx.y;
  const int m = p.cu_rows[j];
  if (p.cu_rows[j + 1] <= m) return;
  const int slot = delta_slot(p, j);
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 7, nt = blockDim.x, nw = nt >> 5;
  const int pos = p.pos[m], group = p.H / p.HK, hk = h / group;
  const int C = 2 * p.HK * p.D + p.H * p.V;
  float* hist = p.hist + static_cast<size_t>(slot) * p.taps * C;
  const size_t now = static_cast<size_t>(pos % p.taps) * C;
  const float* x = p.x + static_cast<size_t>(m) * p.ldx;
  // the first eight columns of this warp are requested before anything else
  float S[NI][4][2] = {};
  const size_t st0 = (static_cast<size_t>(slot) * p.H + h) * p.VP;
  const int cl = (lane >> 3) * 2;
  if (warp * 8 < p.VP) delta_state_io<NI>(p.state + (st0 + warp * 8 + cl) * DP, S, DP, lg, false);

  float sq[2] = {0.f, 0.f};
  for (int d = threadIdx.x; d < DP; d += nt) {
#pragma unroll
    for (int isk = 0; isk < 2; ++isk) {
      float v = 0.f;
      if (d < p.D) {
        const int c = isk * p.HK * p.D + hk * p.D + d, col = (isk ? p.k_off : p.q_off) + hk * p.D + d;
        v = conv_silu(p, hist, c, col, m, 0, pos, C);
        if (h % group == 0) hist[now + c] = x[col];       // ring row of this token: no head of this step reads it
      }
      (isk ? ks : qs)[d] = v;
      sq[isk] += v * v;
    }
  }
  for (int d = threadIdx.x; d < p.VP; d += nt) {
    float v = 0.f;
    if (d < p.V) {
      const int c = 2 * p.HK * p.D + h * p.V + d, col = p.v_off + h * p.V + d;
      v = conv_silu(p, hist, c, col, m, 0, pos, C);
      hist[now + c] = x[col];
    }
    vs[d] = v;
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    sq[i] = warp_sum_f(sq[i]);
    if (lane == 0) red[i][warp] = sq[i];
  }
  __syncthreads();
  if (threadIdx.x < 2) {
    float s = 0.f;
    for (int w = 0; w < nw; ++w) s += red[threadIdx.x][w];
    sum_s[threadIdx.x] = 1.f / sqrtf(s + p.unit_eps) * (threadIdx.x == 0 ? p.q_scale : 1.f);
  }
  __syncthreads();
  for (int d = threadIdx.x; d < DP; d += nt) {
    qs[d] *= sum_s[0];
    ks[d] *= sum_s[1];
  }
  __syncthreads();
  const float beta = sigmoid_f32(x[p.b_off + h]);
  const float g = expf(-expf(p.A_log[h]) * softplus_f32(x[p.a_off + h] + p.dt_bias[h]));
  for (int cb = warp * 8; cb < p.VP; cb += nw * 8) {
    float* st = p.state + (st0 + cb + cl) * DP;
    if (cb != warp * 8) delta_state_io<NI>(st, S, DP, lg, false);
    float o0, o1;
    delta_token<NI>(S, ks, qs, lg, vs[cb + cl], vs[cb + cl + 1], beta, g, o0, o1);
    if (lg == 0) { os[cb + cl] = o0; os[cb + cl + 1] = o1; }
    delta_state_io<NI>(st, S, DP, lg, true);
  }
  __syncthreads();
  // gated norm over V by the whole CTA
  float s2 = 0.f;
  for (int v = threadIdx.x; v < p.V; v += nt) s2 += os[v] * os[v];
  s2 = warp_sum_f(s2);
  if (lane == 0) red[0][warp] = s2;
  __syncthreads();
  s2 = 0.f;
  for (int w = 0; w < nw; ++w) s2 += red[0][w];
  const float r = 1.f / sqrtf(s2 / static_cast<float>(p.V) + p.eps);
  for (int v = threadIdx.x; v < p.V; v += nt)
    operand_store1(p.out, m, p.out_k0 + h * p.V + v, os[v] * r * p.norm_w[v] * silu_f32(x[p.g_off + h * p.V + v]));
}

template <int NI>
static int delta_go(const DeltaParams& p, bool single, cudaStream_t stream) {
  if (single) {
    const int warps = min(8, p.VP / 8);
    const int smem = (2 * NI * 32 + 2 * p.VP) * 4;
    return static_cast<int>(launch(delta_step_kernel<NI>, dim3(p.H, p.nseq), dim3(32 * warps), smem, stream, 0, p));
  }
  const int smem = 2 * kScanRows * (2 * NI * 32 + 36) * 4;
  static bool ready[64];
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return static_cast<int>(cudaErrorInvalidDevice);
  if (!ready[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<NI>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    ready[dev] = true;
  }
  cudaError_t e = launch(delta_prep_kernel, dim3(p.M, (2 * p.HK + p.H + 8) / 8), dim3(256), 0, stream, 0, p);
  if (e == cudaSuccess) e = launch(delta_scan_kernel<NI>, dim3(p.nseq, p.H, (p.VP + 31) / 32), dim3(128), smem, stream, 0, p);
  if (e == cudaSuccess) e = launch(delta_out_kernel, dim3(p.M + p.nseq, (p.H + 7) / 8), dim3(256), 0, stream, 0, p);
  return static_cast<int>(e);
}

}  // namespace saber

extern "C" int saber_delta_launches(int single_row) { return single_row ? 1 : 3; }

extern "C" int saber_delta_launch(const saber::DeltaParams* p, int single_row, cudaStream_t stream) {
  using namespace saber;
  if (p->M <= 0 || p->nseq <= 0 || p->HK <= 0 || p->H % p->HK || p->D > p->DP || (p->VP & 7) || p->V > p->VP || p->VP > 4096 || p->taps < 1)
    return static_cast<int>(cudaErrorInvalidValue);
  switch (p->DP) {
    case 32: return delta_go<1>(*p, single_row != 0, stream);
    case 64: return delta_go<2>(*p, single_row != 0, stream);
    case 96: return delta_go<3>(*p, single_row != 0, stream);
    case 128: return delta_go<4>(*p, single_row != 0, stream);
    case 192: return delta_go<6>(*p, single_row != 0, stream);
    case 256: return delta_go<8>(*p, single_row != 0, stream);
    case 384: return delta_go<12>(*p, single_row != 0, stream);
    case 512: return delta_go<16>(*p, single_row != 0, stream);
    default: return static_cast<int>(cudaErrorInvalidValue);
  }
}
