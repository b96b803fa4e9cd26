// Delta rule with a decay and a removal rate per key channel, free head sizes, fp32 throughout.
//
// Prompt portions (ragged rows, any length), in blocks of four tokens: three launches.
//   prep   decays, unit keys and removal rates, and per block everything that does not depend on the state.  W2 tanh(l) of sixteen
//          tokens is a product on the tensor cores: W2 is bf16, tanh(l) enters as three bf16 parts (24 bits), sums are fp32
//   scan   the recurrence.  Columns of the state are independent, so a warp owns eight value columns for the whole portion: eight
//          lanes split the key dimension, four lane groups take two columns each, the state stays in registers.  With
//          D_ij = w_{j+1} .. w_i (products of decays channel by channel, no quotients), b_i = -rate_i u_i and p_i = u_i^T S_{i-1}:
//              p_i = (u_i D_{i-1,0})^T S_0 + sum_{j<i} (u_i . D_{i-1,j} k_j) v_j + (u_i . D_{i-1,j} b_j) p_j
//              o_i = (r_i D_i0)^T S_0 + sum_{j<=i} (r_i . D_ij k_j) v_j + (r_i . D_ij b_j) p_j
//              S_4 = D_40 S_0 + sum_j (D_4j k_j) v_j^T + (D_4j b_j) p_j^T
//          which is the token-by-token rule written out; the products with S_0 are independent of one another (one shuffle reduction
//          for all), the rest is a triangular recurrence in scalars.  Blocks arrive in shared memory by bulk copies, four in flight.
//   out    norm and gate into the operand of the output linear
// Decoding (one row per sequence): all of it in one launch, a CTA per (head, sequence).
#include "cdelta.h"
#include "launch.cuh"
#include "mla_device.cuh"
#include "ptx_sm100.cuh"
#include "scan_records.cuh"

namespace saber {

// Record of a block and head, contiguous (one bulk copy): u D_{i-1,0} [4][DP] | r D_i0 [4][DP] | D_4j k [4][DP] | D_4j b [4][DP] |
// D_40 [DP] | the dot products: u . D k below the diagonal (6), u . D b (6), 4 unused, r . D k [4][4], r . D b [4][4] (zeros above the
// diagonal).  Missing tokens of the last block have k = r = v = b = u = 0 and decay 1.
constexpr int kCdDots = 32;              // those that are not zero by position
constexpr int kCdTail = 64;                // (records of whole 128 bytes)
__host__ __device__ constexpr int cd_words(int DP) { return 17 * DP + kCdTail; }
__host__ __device__ constexpr int cd_uk(int i, int j) { return kk_at(i, j); }                       // j < i
__host__ __device__ constexpr int cd_ub(int i, int j) { return 6 + kk_at(i, j); }
__host__ __device__ constexpr int cd_rk(int i, int j) { return 12 + i * (i + 1) / 2 + j; }          // j <= i
__host__ __device__ constexpr int cd_rb(int i, int j) { return 22 + i * (i + 1) / 2 + j; }
constexpr int kCdCols = 32;              // value columns of a scan CTA
constexpr int kCdVWords = kBlk * kCdCols;
constexpr float kCdRate = 0.60653065971263342f;  // exp(-1/2)

__device__ __forceinline__ int cd_slot(const CdeltaParams& p, int j) {
  const int s = p.slots[j];
  if (s >= p.n_slots) {
    if (p.err) atomicCAS(p.err, 0u, static_cast<uint32_t>(kErrBadIndex));
    return -1;
  }
  return s;
}
__device__ __forceinline__ bool cd_block_of_slot(const CdeltaParams& p, int slot, int& j, int& c) {
  for (j = 0; j < p.nseq; ++j) {
    const int r0 = p.cu_rows[j], n = p.cu_rows[j + 1] - r0;
    c = slot - block_slot(r0, j, 0);
    if (c >= 0 && c < (n + kBlk - 1) / kBlk) return true;
  }
  return false;
}
__host__ __device__ constexpr int cd_rank_pad(int rank) { return (rank + 15) & ~15; }
// four values of channel c's row of W2, from q (a multiple of 4) on
__device__ __forceinline__ float4 cd_w2(const CdeltaParams& p, int c, int q) {
  const size_t i = static_cast<size_t>(c) * cd_rank_pad(p.rank) + q;
  if (p.w2_f32) return *reinterpret_cast<const float4*>(static_cast<const float*>(p.w2) + i);
  const uint2 u = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p.w2) + i);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xFFFF0000u));
}
__device__ __forceinline__ float cd_decay(float z) { return expf(-kCdRate * sigmoid_f32(z)); }

// Sums over the warp of 32 values a lane: lane n gets the sum of value n (a halving exchange, 31 shuffles).
__device__ __forceinline__ float warp_sums32(float (&v)[32], int lane) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = (lane & o) != 0;
#pragma unroll
    for (int e = 0; e < o; ++e) {
      const float keep = up ? v[o + e] : v[e], give = up ? v[e] : v[o + e];
      v[e] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
  return v[0];
}

// A store that no load has to wait for (the caller never reads what it writes).
__device__ __forceinline__ void store_f32(float* p, float v) { asm volatile("st.global.f32 [%0], %1;" ::"l"(p), "f"(v)); }

// The same over eight lanes and values (7 shuffles): lane lg of its eight gets value lg in v[0].
__device__ __forceinline__ void scan_sums8(float (&v)[8], int lg) {
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) {
    const bool up = (lg & o) != 0;
#pragma unroll
    for (int e = 0; e < o; ++e) {
      const float keep = up ? v[o + e] : v[e], give = up ? v[e] : v[o + e];
      v[e] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
}

// Records of a block (rows live tokens from x on) and head h, by a warp.  mid(): what comes between the loads of the head's projections
// and their use.  z(i, c, out): the arguments of the decays of channel c (32 i + lane
// inside the head) of the four tokens, w0 not yet in them.
template <int NI, typename Mid, typename Z>
__device__ __forceinline__ void cd_records(const CdeltaParams& p, const float* x, int rows, int h, int slot, int lane, const Mid& mid, const Z& zget) {
  constexpr int DP = NI * 32;
  constexpr bool kHold = NI <= 4;                  // every load of the block at once, else of 32 channels at a time
  const float* xr[kBlk];                           // (rows past the live ones repeat the last, channels past the head its first: not used)
#pragma unroll
  for (int r = 0; r < kBlk; ++r) xr[r] = x + static_cast<size_t>(min(r, rows - 1)) * p.ldx + h * p.D;
  float kh[kHold ? NI : 1][kBlk], ah[kHold ? NI : 1][kBlk], rh[kHold ? NI : 1][kBlk], vh[kHold ? NI : 1][kBlk], w0[kHold ? NI : 1], inv[kBlk];
  if constexpr (kHold) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int dc = i * 32 + lane < p.D ? i * 32 + lane : 0;
#pragma unroll
      for (int r = 0; r < kBlk; ++r) {
        kh[i][r] = xr[r][p.k_off + dc];
        ah[i][r] = xr[r][p.a_off + dc];
        rh[i][r] = xr[r][p.r_off + dc];
        vh[i][r] = xr[r][p.v_off + dc];
      }
      w0[i] = p.w0[h * p.D + dc];
    }
  }
  mid();
#pragma unroll
  for (int r = 0; r < kBlk; ++r) inv[r] = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = i * 32 + lane, dc = d < p.D ? d : 0;
#pragma unroll
    for (int r = 0; r < kBlk; ++r) {
      const float k = kHold ? kh[kHold ? i : 0][r] : xr[r][p.k_off + dc];
      inv[r] = fmaf(d < p.D ? k : 0.f, k, inv[r]);
    }
  }
#pragma unroll
  for (int r = 0; r < kBlk; ++r) inv[r] = 1.f / sqrtf(warp_sum_f(inv[r]) + p.unit_eps);
  float* o = p.rec + (static_cast<size_t>(slot) * p.H + h) * cd_words(DP);
  float dots[kCdDots];
#pragma unroll
  for (int e = 0; e < kCdDots; ++e) dots[e] = 0.f;
  constexpr int kUnroll = kHold ? NI : 1;
#pragma unroll kUnroll
  for (int i = 0; i < NI; ++i) {
    const int d = i * 32 + lane, c = h * p.D + d, dc = d < p.D ? d : 0;
    float w[kBlk], k[kBlk], b[kBlk], u[kBlk], rr[kBlk], z[kBlk];
    const bool in = d < p.D;
    if constexpr (!kHold) {
      w0[0] = p.w0[h * p.D + dc];
#pragma unroll
      for (int r = 0; r < kBlk; ++r) {
        kh[0][r] = xr[r][p.k_off + dc];
        ah[0][r] = xr[r][p.a_off + dc];
        rh[0][r] = xr[r][p.r_off + dc];
      }
    }
    zget(i, in ? c : -1, z);
#pragma unroll
    for (int r = 0; r < kBlk; ++r) {
      const bool live = in && r < rows;
      const int ih = kHold ? i : 0;
      const float dec = cd_decay(z[r] + w0[ih]), rate = sigmoid_f32(ah[ih][r]);
      w[r] = live ? dec : 1.f;
      k[r] = live ? kh[ih][r] : 0.f;
      u[r] = k[r] * inv[r];
      b[r] = -rate * u[r];
      rr[r] = live ? rh[ih][r] : 0.f;
    }
    // row t of the triangle against j = t, t - 1, ..: the product of the decays between them grows by one at a time
#pragma unroll
    for (int t = 0; t < kBlk; ++t) {
      float g = 1.f;                               // D_{t-1,j}
      dots[cd_rk(t, t)] = fmaf(rr[t], k[t], dots[cd_rk(t, t)]);
      dots[cd_rb(t, t)] = fmaf(rr[t], b[t], dots[cd_rb(t, t)]);
      const float rw = rr[t] * w[t];
#pragma unroll
      for (int jj = t - 1; jj >= 0; --jj) {
        const float gk = g * k[jj], gb = g * b[jj];
        dots[cd_uk(t, jj)] = fmaf(u[t], gk, dots[cd_uk(t, jj)]);
        dots[cd_ub(t, jj)] = fmaf(u[t], gb, dots[cd_ub(t, jj)]);
        dots[cd_rk(t, jj)] = fmaf(rw, gk, dots[cd_rk(t, jj)]);
        dots[cd_rb(t, jj)] = fmaf(rw, gb, dots[cd_rb(t, jj)]);
        g *= w[jj];
      }
      o[t * DP + d] = u[t] * g;                    // g is D_{t-1,0} now
      o[(kBlk + t) * DP + d] = rw * g;
    }
    float g = 1.f;
#pragma unroll
    for (int t = kBlk - 1; t >= 0; --t) {
      o[(2 * kBlk + t) * DP + d] = g * k[t];
      o[(3 * kBlk + t) * DP + d] = g * b[t];
      g *= w[t];
    }
    o[4 * kBlk * DP + d] = g;
  }
  const float mine = warp_sums32(dots, lane);
  {
    float* tail = o + (4 * kBlk + 1) * DP;
    const int e = lane < 12 ? 0 : lane < 22 ? lane - 12 : lane - 22;                    // r . D k and r . D b in rows of four
    const int row = e >= 6 ? 3 : e >= 3 ? 2 : e >= 1 ? 1 : 0, at = 4 * row + e - row * (row + 1) / 2;
    tail[lane < 12 ? lane : lane < 22 ? 16 + at : 32 + at] = mine;
    if (lane < 12) tail[(lane < 6 ? 16 : 32) + (lane % 6 < 3 ? lane % 6 + 1 : lane % 6 < 5 ? lane % 6 + 3 : 11)] = 0.f;      // 1, 2, 3, 6, 7, 11
  }
  const int groups = (p.VP + kCdCols - 1) / kCdCols;
#pragma unroll
  for (int gr = 0; gr < NI; ++gr) {                // (never more than the key's pieces of 32)
    if (gr >= groups) break;
    const int d = gr * kCdCols + lane;
    float* vo = p.vb + ((static_cast<size_t>(slot) * p.H + h) * groups + gr) * kCdVWords + lane;
#pragma unroll
    for (int r = 0; r < kBlk; ++r) {
      const float v = kHold ? vh[kHold ? gr : 0][r] : xr[r][p.v_off + (d < p.D ? d : 0)];
      vo[r * kCdCols] = d < p.D && r < rows ? v : 0.f;
    }
  }
}

// grid (blocks, ceil(H / 4)), 128 threads; a warp per (block, head); shared memory: tanh of the four tokens' `rank` values
template <int NI>
__global__ void __launch_bounds__(128) cdelta_prep_kernel(const __grid_constant__ CdeltaParams p) {
  pdl_wait();
  extern __shared__ float4 sm4[];                  // [rank, padded] values of four tokens
  const int lane = threadIdx.x & 31, h = blockIdx.y * 4 + (threadIdx.x >> 5), RK = cd_rank_pad(p.rank);
  int j, blk;
  if (!cd_block_of_slot(p, blockIdx.x, j, blk)) return;
  if (cd_slot(p, j) < 0) return;
  const int m = p.cu_rows[j] + blk * kBlk, rows = min(kBlk, p.cu_rows[j + 1] - m);
  const float* x = p.x + static_cast<size_t>(m) * p.ldx;
  for (int q = threadIdx.x; q < RK; q += 128) {
    float t[kBlk];
#pragma unroll
    for (int r = 0; r < kBlk; ++r) t[r] = r < rows && q < p.rank ? tanhf(x[static_cast<size_t>(r) * p.ldx + p.l_off + q]) : 0.f;
    sm4[q] = make_float4(t[0], t[1], t[2], t[3]);
  }
  __syncthreads();
  if (h >= p.H) return;
  cd_records<NI>(p, x, rows, h, blockIdx.x, lane, [] {}, [&](int, int c, float (&z)[kBlk]) {
#pragma unroll
    for (int r = 0; r < kBlk; ++r) z[r] = 0.f;
    if (c < 0) return;
#pragma unroll 2
    for (int q = 0; q < RK; q += 4) {
      const float4 f = cd_w2(p, c, q);
      const float fa[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float4 t = sm4[q + e];
        z[0] = fmaf(fa[e], t.x, z[0]);
        z[1] = fmaf(fa[e], t.y, z[1]);
        z[2] = fmaf(fa[e], t.z, z[2]);
        z[3] = fmaf(fa[e], t.w, z[3]);
      }
    }
  });
}

constexpr int kCdMmaRank = 256;          // largest padded rank of the tensor-core form
constexpr int kCdMmaHeads = 4;           // heads of a CTA

// The same for bf16 W2, grid (ceil(blocks / 4), ceil(H / kCdMmaHeads)), 128 threads: four blocks (sixteen tokens), a warp per block; the
// product W2 tanh(l) of a head by all four warps.  Shared memory: tanh in three parts [3][16][RK + 8] bf16, products [16][DP + 4].
template <int NI>
__global__ void __launch_bounds__(128) cdelta_prep_mma_kernel(const __grid_constant__ CdeltaParams p) {
  pdl_wait();
  constexpr int DP = NI * 32, ZS = DP + 4;
  extern __shared__ float4 sm4[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, RK = cd_rank_pad(p.rank);
  const uint32_t ts = smem_u32(sm4), t_row = static_cast<uint32_t>(RK + 8) * 2u, t_part = 16u * t_row;
  float* zs = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(sm4) + 3 * t_part);
  const int slot = blockIdx.x * 4 + warp;
  int j, blk, rows = 0;
  const float* x = p.x;
  if (cd_block_of_slot(p, slot, j, blk) && cd_slot(p, j) >= 0) {
    const int m = p.cu_rows[j] + blk * kBlk;
    rows = min(kBlk, p.cu_rows[j + 1] - m);
    x += static_cast<size_t>(m) * p.ldx;
  }
  if (__syncthreads_or(rows) == 0) return;
#pragma unroll
  for (int r = 0; r < kBlk; ++r)
    for (int q = lane; q < RK; q += 32) {
      float t = r < rows && q < p.rank ? tanhf(x[static_cast<size_t>(r) * p.ldx + p.l_off + q]) : 0.f;
#pragma unroll
      for (int part = 0; part < 3; ++part) {
        const __nv_bfloat16 v = __float2bfloat16(t);
        asm volatile("st.shared.b16 [%0], %1;" ::"r"(ts + part * t_part + (warp * kBlk + r) * t_row + q * 2), "h"(__bfloat16_as_ushort(v)) : "memory");
        t -= __bfloat162float(v);
      }
    }
  const uint32_t a_row = ts + static_cast<uint32_t>(lane & 15) * t_row + ((lane >> 4) << 4);
  const __nv_bfloat16* w2 = static_cast<const __nv_bfloat16*>(p.w2);
  const int h1 = min(p.H, (static_cast<int>(blockIdx.y) + 1) * kCdMmaHeads);
  for (int h = blockIdx.y * kCdMmaHeads; h < h1; ++h) {
    auto product = [&] {
      named_bar_sync(1, 128);                        // (tanh is there; the products of the head before are read)
      float acc[NI][4] = {};
      const __nv_bfloat16* wr[NI];
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int d = (warp * NI + i) * 8 + (lane >> 2);
        wr[i] = w2 + static_cast<size_t>(h * p.D + (d < p.D ? d : 0)) * RK + (lane & 3) * 2;
      }
      uint32_t nb[NI][2];                            // the next step's pieces of W2
      auto fetch = [&](int k0) {
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          nb[i][0] = *reinterpret_cast<const uint32_t*>(wr[i] + k0);
          nb[i][1] = *reinterpret_cast<const uint32_t*>(wr[i] + k0 + 8);
        }
      };
      fetch(0);
      for (int k0 = 0; k0 < RK; k0 += 16) {
        uint32_t a[3][4], bb[NI][2];
#pragma unroll
        for (int i = 0; i < NI; ++i) { bb[i][0] = nb[i][0]; bb[i][1] = nb[i][1]; }
        if (k0 + 16 < RK) fetch(k0 + 16);
#pragma unroll
        for (int part = 0; part < 3; ++part) ldsm4(a[part], a_row + part * t_part + k0 * 2);
#pragma unroll
        for (int i = 0; i < NI; ++i)                 // (channels past the head: numbers that nothing reads)
#pragma unroll
          for (int part = 2; part >= 0; --part) mma16816(acc[i], a[part], bb[i][0], bb[i][1]);
      }
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        float* d = zs + (lane >> 2) * ZS + (warp * NI + i) * 8 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(d) = make_float2(acc[i][0], acc[i][1]);
        *reinterpret_cast<float2*>(d + 8 * ZS) = make_float2(acc[i][2], acc[i][3]);
      }
      named_bar_sync(1, 128);                        // (warps with and without a block meet here)
    };
    if (rows > 0)
      cd_records<NI>(p, x, rows, h, slot, lane, product, [&](int i, int, float (&z)[kBlk]) {
#pragma unroll
        for (int r = 0; r < kBlk; ++r) z[r] = zs[(warp * kBlk + r) * ZS + i * 32 + lane];
      });
    else product();
  }
}

constexpr int kCdStages = 4;             // blocks of four tokens in flight
constexpr int kCdScanThreads = 160;

// grid (nseq, H, ceil(VP / 32)), 160 threads: four warps of eight value columns, each at its own pace, and a warp whose first lane
// keeps the copies going
template <int NI>
__global__ void __launch_bounds__(kCdScanThreads) cdelta_scan_kernel(const __grid_constant__ CdeltaParams p) {
  constexpr int DP = NI * 32;
  constexpr int kRec = cd_words(DP);
  constexpr int kStageWords = kRec + kCdVWords;
  extern __shared__ float4 sm4[];
  float* sm = reinterpret_cast<float*>(sm4);
  __shared__ uint64_t bars[2 * kCdStages];
  pdl_wait();
  const int j = blockIdx.x, h = blockIdx.y;
  const int r0 = p.cu_rows[j], n = p.cu_rows[j + 1] - r0;
  if (n <= 0) return;
  const int slot = cd_slot(p, j);
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 7;
  const int vb = blockIdx.z * kCdCols, groups = (p.VP + kCdCols - 1) / kCdCols;
  const int cl = warp * 8 + (lane >> 3) * 2;       // columns inside the CTA's 32
  const bool on = vb + warp * 8 < p.VP;            // VP is a multiple of 8
  const int blocks = (n + kBlk - 1) / kBlk;
  const uint32_t bar = smem_u32(bars), bar_free = bar + 8 * kCdStages;
  const uint32_t sm_u = smem_u32(sm);
  if (threadIdx.x == 0) {
    for (int i = 0; i < kCdStages; ++i) {
      mbar_init(bar + 8 * i, 1);
      mbar_init(bar_free + 8 * i, 4);
    }
    mbar_init_fence();
  }
  __syncthreads();
  if (warp == 4) {                                 // ---- copies
    if (lane == 0) {
      const size_t bs0 = static_cast<size_t>(block_slot(r0, j, 0));
      const float* rec = p.rec + (bs0 * p.H + h) * kRec;
      const float* vr = p.vb + ((bs0 * p.H + h) * groups + blockIdx.z) * kCdVWords;
      const size_t rec_step = static_cast<size_t>(p.H) * kRec, v_step = static_cast<size_t>(p.H) * groups * kCdVWords;
      int blk = 0;
      for (; blk < blocks; ++blk) {
        const int s = blk % kCdStages;
        if (blk >= kCdStages && !mbar_wait(bar_free + 8 * s, ((blk / kCdStages) & 1) ^ 1, p.err, kErrWaitEmpty)) break;
        mbar_arrive_expect_tx(bar + 8 * s, kStageWords * 4);
        bulk_g2s(sm_u + s * kStageWords * 4, rec + blk * rec_step, kRec * 4, bar + 8 * s);
        bulk_g2s(sm_u + (s * kStageWords + kRec) * 4, vr + blk * v_step, kCdVWords * 4, bar + 8 * s);
      }
      for (int i = max(0, blk - kCdStages); i < blk; ++i)          // the CTA does not leave before its copies have landed
        mbar_wait(bar + 8 * (i % kCdStages), (i / kCdStages) & 1, p.err, kErrWaitDrain);
    }
    return;
  }
  f32x2 S[NI][2][2] = {};                          // [32 keys][pair of keys][column]
  float* st = p.state + ((static_cast<size_t>(slot) * p.H + h) * p.VP + vb + cl) * DP;
  if (on) {
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(st + static_cast<size_t>(c) * DP + i * 32 + lg * 4);
        S[i][0][c] = f.x;
        S[i][1][c] = f.y;
      }
  }
  const int tok = lg >> 1, col = lg & 1;           // whose values this lane keeps
  float* out = p.o + (static_cast<size_t>(r0 + tok) * p.H + h) * p.VP + vb + cl + col;
  const size_t out_step = static_cast<size_t>(kBlk) * p.H * p.VP;
  for (int blk = 0; blk < blocks; ++blk) {
    const int s = blk % kCdStages;
    if (!mbar_wait(bar + 8 * s, (blk / kCdStages) & 1, p.err, kErrWaitFull)) break;
    const float* b = sm + s * kStageWords;
    const float* vrec = b + kRec;
    if (on) {
      float sk[kBlk][2], sq[8];                    // [token][column]
#pragma unroll
      for (int r = 0; r < kBlk; ++r) {
        f32x2 a[2] = {}, c[2] = {};
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          const ulonglong2 u4 = *reinterpret_cast<const ulonglong2*>(b + r * DP + i * 32 + lg * 4);
          const ulonglong2 r4 = *reinterpret_cast<const ulonglong2*>(b + (kBlk + r) * DP + i * 32 + lg * 4);
#pragma unroll
          for (int v = 0; v < 2; ++v) {
            a[v] = fma_f2(S[i][0][v], u4.x, a[v]);
            a[v] = fma_f2(S[i][1][v], u4.y, a[v]);
            c[v] = fma_f2(S[i][0][v], r4.x, c[v]);
            c[v] = fma_f2(S[i][1][v], r4.y, c[v]);
          }
        }
#pragma unroll
        for (int v = 0; v < 2; ++v) {
          const float2 e = unpack_f2(a[v]), f = unpack_f2(c[v]);
          sk[r][v] = e.x + e.y;
          sq[r * 2 + v] = f.x + f.y;
        }
      }
#pragma unroll
      for (int o = 1; o < 8; o <<= 1)
#pragma unroll
        for (int r = 0; r < kBlk; ++r)
#pragma unroll
          for (int v = 0; v < 2; ++v) sk[r][v] += __shfl_xor_sync(0xffffffffu, sk[r][v], o);
      scan_sums8(sq, lg);
      const float* tail = b + (4 * kBlk + 1) * DP;
      float pr[48], held[kBlk][2], val[kBlk][2];
#pragma unroll
      for (int e = 0; e < 48; e += 4)
        if (e != 12) *reinterpret_cast<float4*>(pr + e) = *reinterpret_cast<const float4*>(tail + e);
#pragma unroll
      for (int i = 0; i < kBlk; ++i) {
        const float2 v = *reinterpret_cast<const float2*>(vrec + i * kCdCols + cl);
        val[i][0] = v.x;
        val[i][1] = v.y;
      }
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < kBlk; ++i) {
#pragma unroll
        for (int v = 0; v < 2; ++v) {
          float a = sk[i][v];
#pragma unroll
          for (int jj = 0; jj < i; ++jj) a = fmaf(pr[cd_uk(i, jj)], val[jj][v], a);      // (what does not wait for `held` first)
#pragma unroll
          for (int jj = 0; jj < i; ++jj) a = fmaf(pr[cd_ub(i, jj)], held[jj][v], a);
          held[i][v] = a;
        }
        float t = sq[0];
#pragma unroll
        for (int jj = 0; jj <= i; ++jj)
          t = fmaf(pr[16 + 4 * i + jj], col ? val[jj][1] : val[jj][0], fmaf(pr[32 + 4 * i + jj], col ? held[jj][1] : held[jj][0], t));
        o = tok == i ? t : o;
      }
      if (blk * kBlk + tok < n) store_f32(out + blk * out_step, o);
      f32x2 v2[kBlk][2], p2[kBlk][2];
#pragma unroll
      for (int r = 0; r < kBlk; ++r)
#pragma unroll
        for (int v = 0; v < 2; ++v) {
          v2[r][v] = pack_f2(val[r][v], val[r][v]);
          p2[r][v] = pack_f2(held[r][v], held[r][v]);
        }
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const ulonglong2 g4 = *reinterpret_cast<const ulonglong2*>(b + 4 * kBlk * DP + i * 32 + lg * 4);
#pragma unroll
        for (int v = 0; v < 2; ++v) {
          S[i][0][v] = mul_f2(S[i][0][v], g4.x);
          S[i][1][v] = mul_f2(S[i][1][v], g4.y);
        }
#pragma unroll
        for (int r = 0; r < kBlk; ++r) {
          const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(b + (2 * kBlk + r) * DP + i * 32 + lg * 4);
          const ulonglong2 b4 = *reinterpret_cast<const ulonglong2*>(b + (3 * kBlk + r) * DP + i * 32 + lg * 4);
#pragma unroll
          for (int v = 0; v < 2; ++v) {
            S[i][0][v] = fma_f2(p2[r][v], b4.x, fma_f2(v2[r][v], k4.x, S[i][0][v]));
            S[i][1][v] = fma_f2(p2[r][v], b4.y, fma_f2(v2[r][v], k4.y, S[i][1][v]));
          }
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(bar_free + 8 * s);  // this warp is done with the stage
  }
  if (on) {
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
      for (int i = 0; i < NI; ++i)
        *reinterpret_cast<ulonglong2*>(st + static_cast<size_t>(c) * DP + i * 32 + lg * 4) = make_ulonglong2(S[i][0][c], S[i][1][c]);
  }
}

// grid (M, ceil(H / 8)): a warp per (row, head)
__global__ void __launch_bounds__(256) cdelta_out_kernel(const __grid_constant__ CdeltaParams p) {
  pdl_wait();
  const int lane = threadIdx.x & 31, m = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (h >= p.H || seq_of_row(p.cu_rows, p.nseq, m) < 0) return;
  const float* o = p.o + (static_cast<size_t>(m) * p.H + h) * p.VP;
  const float* g = p.x + static_cast<size_t>(m) * p.ldx + p.g_off + h * p.D;
  const float* w = p.norm_w + h * p.D;
  float sq = 0.f;
  for (int v = lane; v < p.D; v += 32) sq = fmaf(o[v], o[v], sq);
  const float r = p.out_scale / sqrtf(warp_sum_f(sq) / static_cast<float>(p.D) + p.eps);
  if ((p.D & 3) == 0) {                            // (columns of a projection start at multiples of 8)
    for (int v = lane * 4; v < p.D; v += 128) {
      const float4 a = *reinterpret_cast<const float4*>(o + v), b = *reinterpret_cast<const float4*>(g + v), c = *reinterpret_cast<const float4*>(w + v);
      operand_store4(p.out, m, p.out_k0 + h * p.D + v,
                     make_float4(a.x * r * c.x * sigmoid_f32(b.x), a.y * r * c.y * sigmoid_f32(b.y), a.z * r * c.z * sigmoid_f32(b.z), a.w * r * c.w * sigmoid_f32(b.w)));
    }
    return;
  }
  for (int v = lane; v < p.D; v += 32) operand_store1(p.out, m, p.out_k0 + h * p.D + v, o[v] * r * w[v] * sigmoid_f32(g[v]));
}

template <int NI>
__device__ __forceinline__ void cd_state_io(float* st, float (&S)[NI][4][2], int lg, bool store) {
#pragma unroll
  for (int c = 0; c < 2; ++c)
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      float4* a = reinterpret_cast<float4*>(st + static_cast<size_t>(c) * (NI * 32) + i * 32 + lg * 4);
      if (store) {
        *a = make_float4(S[i][0][c], S[i][1][c], S[i][2][c], S[i][3][c]);
      } else {
        const float4 f = *a;
        S[i][0][c] = f.x; S[i][1][c] = f.y; S[i][2][c] = f.z; S[i][3][c] = f.w;
      }
    }
}

constexpr int kCdParts = 4;              // parts of the rank that a channel's decay is summed in

// One row per sequence: grid (H, nseq), 32 * min(8, VP / 8) threads.
template <int NI>
__global__ void __launch_bounds__(256) cdelta_step_kernel(const __grid_constant__ CdeltaParams p) {
  pdl_trigger();
  extern __shared__ float4 sm4[];
  constexpr int DP = NI * 32;
  float* us = reinterpret_cast<float*>(sm4);       // DP: unit key, then of the same size each
  float* rs = us + DP;                             // r w
  float* ws = rs + DP;                             // decay
  float* bs = ws + DP;                             // -rate u
  float* ks = bs + DP;                             // key
  float* zs = ks + DP;                             // [kCdParts][DP]
  float* ts = zs + kCdParts * DP;                  // [rank, padded] tanh of the shared values
  float* vs = ts + cd_rank_pad(p.rank);            // VP
  float* os = vs + p.VP;                           // VP
  __shared__ float red[3][8];
  const int h = blockIdx.x, j = blockIdx.y;
  const int m = p.cu_rows[j];
  const bool live = p.cu_rows[j + 1] > m;
  const int slot = live ? cd_slot(p, j) : -1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 7, nt = blockDim.x, nw = nt >> 5;
  // the first eight columns of this warp are requested before anything else (only an earlier step wrote them)
  float S[NI][4][2] = {};
  const size_t st0 = (static_cast<size_t>(max(slot, 0)) * p.H + h) * p.VP;
  const int cl = (lane >> 3) * 2;
  if (slot >= 0 && warp * 8 < p.VP) cd_state_io<NI>(p.state + (st0 + warp * 8 + cl) * DP, S, lg, false);
  pdl_wait();
  if (slot < 0) return;
  const float* x = p.x + static_cast<size_t>(m) * p.ldx;
  for (int q = threadIdx.x; q < cd_rank_pad(p.rank); q += nt) ts[q] = q < p.rank ? tanhf(x[p.l_off + q]) : 0.f;
  float sum[3] = {0.f, 0.f, 0.f};                  // k . k, r . k, r . rate k
  for (int d = threadIdx.x; d < DP; d += nt) {
    float k = 0.f, r = 0.f, a = 0.f;
    if (d < p.D) {
      const int c = h * p.D + d;
      k = x[p.k_off + c];
      r = x[p.r_off + c];
      a = sigmoid_f32(x[p.a_off + c]);
    }
    ks[d] = k;
    rs[d] = r;
    bs[d] = -a * k;
    sum[0] = fmaf(k, k, sum[0]);
    sum[1] = fmaf(r, k, sum[1]);
    sum[2] = fmaf(r * a, k, sum[2]);
  }
  for (int d = threadIdx.x; d < p.VP; d += nt) vs[d] = d < p.D ? x[p.v_off + h * p.D + d] : 0.f;
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    sum[i] = warp_sum_f(sum[i]);
    if (lane == 0) red[i][warp] = sum[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    sum[i] = 0.f;
    for (int w = 0; w < nw; ++w) sum[i] += red[i][w];
  }
  const float inv = 1.f / sqrtf(sum[0] + p.unit_eps), rk = sum[1], rb = -inv * sum[2];
  const int RK = cd_rank_pad(p.rank), per = RK / kCdParts;
  for (int i = threadIdx.x; i < kCdParts * DP; i += nt) {
    const int part = i / DP, d = i - part * DP;
    float z = 0.f;
    if (d < p.D) {
#pragma unroll 6
      for (int q = part * per; q < (part + 1) * per; q += 4) {
        const float4 f = cd_w2(p, h * p.D + d, q), t = *reinterpret_cast<const float4*>(ts + q);
        z = fmaf(f.x, t.x, fmaf(f.y, t.y, fmaf(f.z, t.z, fmaf(f.w, t.w, z))));
      }
    }
    zs[i] = z;
  }
  __syncthreads();
  for (int d = threadIdx.x; d < DP; d += nt) {
    float z = d < p.D ? p.w0[h * p.D + d] : 0.f;
#pragma unroll
    for (int part = 0; part < kCdParts; ++part) z += zs[part * DP + d];
    const float w = cd_decay(z);
    ws[d] = w;
    us[d] = ks[d] * inv;
    rs[d] *= w;
    bs[d] *= inv;
  }
  __syncthreads();
  for (int cb = warp * 8; cb < p.VP; cb += nw * 8) {
    float* st = p.state + (st0 + cb + cl) * DP;
    if (cb != warp * 8) cd_state_io<NI>(st, S, lg, false);
    float sk0 = 0.f, sk1 = 0.f, sq0 = 0.f, sq1 = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const float4 u4 = *reinterpret_cast<const float4*>(us + i * 32 + lg * 4), r4 = *reinterpret_cast<const float4*>(rs + i * 32 + lg * 4);
      const float ua[4] = {u4.x, u4.y, u4.z, u4.w}, ra[4] = {r4.x, r4.y, r4.z, r4.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        sk0 = fmaf(S[i][e][0], ua[e], sk0);
        sk1 = fmaf(S[i][e][1], ua[e], sk1);
        sq0 = fmaf(S[i][e][0], ra[e], sq0);
        sq1 = fmaf(S[i][e][1], ra[e], sq1);
      }
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) {
      sk0 += __shfl_xor_sync(0xffffffffu, sk0, o);
      sk1 += __shfl_xor_sync(0xffffffffu, sk1, o);
      sq0 += __shfl_xor_sync(0xffffffffu, sq0, o);
      sq1 += __shfl_xor_sync(0xffffffffu, sq1, o);
    }
    const float v0 = vs[cb + cl], v1 = vs[cb + cl + 1];
    if (lg == 0) {
      os[cb + cl] = fmaf(rk, v0, fmaf(rb, sk0, sq0));
      os[cb + cl + 1] = fmaf(rk, v1, fmaf(rb, sk1, sq1));
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const float4 w4 = *reinterpret_cast<const float4*>(ws + i * 32 + lg * 4), k4 = *reinterpret_cast<const float4*>(ks + i * 32 + lg * 4),
                   b4 = *reinterpret_cast<const float4*>(bs + i * 32 + lg * 4);
      const float wa[4] = {w4.x, w4.y, w4.z, w4.w}, ka[4] = {k4.x, k4.y, k4.z, k4.w}, ba[4] = {b4.x, b4.y, b4.z, b4.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        S[i][e][0] = fmaf(wa[e], S[i][e][0], fmaf(ba[e], sk0, ka[e] * v0));
        S[i][e][1] = fmaf(wa[e], S[i][e][1], fmaf(ba[e], sk1, ka[e] * v1));
      }
    }
    cd_state_io<NI>(st, S, lg, true);
  }
  __syncthreads();
  float s2 = 0.f;
  for (int v = threadIdx.x; v < p.D; v += nt) s2 = fmaf(os[v], os[v], s2);
  s2 = warp_sum_f(s2);
  if (lane == 0) red[0][warp] = s2;
  __syncthreads();
  s2 = 0.f;
  for (int w = 0; w < nw; ++w) s2 += red[0][w];
  const float r = p.out_scale / sqrtf(s2 / static_cast<float>(p.D) + p.eps);
  for (int v = threadIdx.x; v < p.D; v += nt)
    operand_store1(p.out, m, p.out_k0 + h * p.D + v, os[v] * r * p.norm_w[h * p.D + v] * sigmoid_f32(x[p.g_off + h * p.D + v]));
}

template <typename Kernel>
static cudaError_t cd_allow(Kernel kernel, bool (&ready)[64], int smem) {
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return cudaErrorInvalidDevice;
  if (ready[dev]) return cudaSuccess;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  ready[dev] = e == cudaSuccess;
  return e;
}

template <int NJ>
static int cdelta_go(const CdeltaParams& p, bool single, cudaStream_t stream) {
  constexpr int NI = NJ * 2, DP = NJ * 64;
  if (single) {
    const int warps = min(8, p.VP / 8);
    const int smem = ((5 + kCdParts) * DP + cd_rank_pad(p.rank) + 2 * p.VP) * 4;
    return static_cast<int>(launch(cdelta_step_kernel<NI>, dim3(p.H, p.nseq), dim3(32 * warps), smem, stream, 2, p));
  }
  static bool ready[64];
  constexpr int smem = kCdStages * (cd_words(DP) + kCdVWords) * 4;
  cudaError_t e = cd_allow(cdelta_scan_kernel<NI>, ready, smem);
  if (e != cudaSuccess) return static_cast<int>(e);
  const int blocks = p.M / kBlk + p.nseq, RK = cd_rank_pad(p.rank);
  bool mma = false;
  if constexpr (DP <= 256) mma = !p.w2_f32 && RK <= kCdMmaRank;
  if constexpr (DP <= 256)
    if (mma)
      e = launch(cdelta_prep_mma_kernel<NI>, dim3((blocks + 3) / 4, (p.H + kCdMmaHeads - 1) / kCdMmaHeads), dim3(128), 3 * 16 * (RK + 8) * 2 + 16 * (DP + 4) * 4, stream, 0, p);
  if (!mma) e = launch(cdelta_prep_kernel<NI>, dim3(blocks, (p.H + 3) / 4), dim3(128), RK * 16, stream, 0, p);
  if (e == cudaSuccess) e = launch(cdelta_scan_kernel<NI>, dim3(p.nseq, p.H, (p.VP + kCdCols - 1) / kCdCols), dim3(kCdScanThreads), smem, stream, 0, p);
  if (e == cudaSuccess) e = launch(cdelta_out_kernel, dim3(p.M, (p.H + 7) / 8), dim3(256), 0, stream, 0, p);
  return static_cast<int>(e);
}

}  // namespace saber

extern "C" int saber_cdelta_launches(int single_row) { return single_row ? 1 : 3; }

extern "C" int saber_cdelta_launch(const saber::CdeltaParams* p, int single_row, cudaStream_t stream) {
  using namespace saber;
  if (p->M <= 0 || p->nseq <= 0 || p->H <= 0 || p->D < 1 || p->D > p->DP || p->D > p->VP || (p->VP & 7) || p->VP > 512 || p->rank < 1 || p->rank > 2048 ||
      p->w2 == nullptr || p->state == nullptr || (!single_row && (p->rec == nullptr || p->vb == nullptr || p->o == nullptr)))
    return static_cast<int>(cudaErrorInvalidValue);
  switch (p->DP) {
    case 64: return cdelta_go<1>(*p, single_row != 0, stream);
    case 128: return cdelta_go<2>(*p, single_row != 0, stream);
    case 192: return cdelta_go<3>(*p, single_row != 0, stream);
    case 256: return cdelta_go<4>(*p, single_row != 0, stream);
    case 384: return cdelta_go<6>(*p, single_row != 0, stream);
    case 512: return cdelta_go<8>(*p, single_row != 0, stream);
    default: return static_cast<int>(cudaErrorInvalidValue);
  }
}
