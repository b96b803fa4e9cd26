// Gated delta rule with free head sizes, fp32 throughout.
//
// Prompt portions (ragged rows, any length), in blocks of four tokens: three launches.
//   prep   convolution, silu, unit norms, beta and decay, and per block the dot products k_j . k_i and k_j . q_i
//   scan   the recurrence.  Columns of the state are independent, so a warp owns four value columns for the
//          whole portion: sixteen lanes split the key dimension, two lane groups take two columns each, the state
//          stays in registers.  A block of four tokens needs the products of its keys and queries with the state
//          at its start only, S_0^T k_i and S_0^T q_i (independent of one another, one shuffle reduction for
//          all); the rest is a triangular recurrence in scalars.  With G_i = g_1 .. g_i and
//          D_ij = g_{j+1} .. g_i (products, no quotients):
//              u_i = beta_i (v_i - G_i S_0^T k_i - sum_{j<i} D_ij (k_j . k_i) u_j)
//              o_i = G_i S_0^T q_i + sum_{j<=i} D_ij (k_j . q_i) u_j
//              S_4 = G_4 S_0 + sum_j D_4j k_j u_j^T
//          which is the token-by-token rule written out; a block with fewer tokens is filled up with
//          k = q = v = beta = 0, g = 1.  Blocks arrive in shared memory by bulk copies, four in flight.
//   out    gated norm into the operand of the output linear; the convolution inputs go to the ring
// Decoding (one row per sequence): all of it in one launch, a CTA per (head, sequence).
#include "delta.h"
#include "launch.cuh"
#include "ptx_sm100.cuh"
#include "scan_records.cuh"

namespace saber {

// slot of a sequence (< 0: none)
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

__device__ __forceinline__ bool block_of_slot(const DeltaParams& p, int slot, int& j, int& c) {
  for (j = 0; j < p.nseq; ++j) {
    const int r0 = p.cu_rows[j], n = p.cu_rows[j + 1] - r0;
    c = slot - ((r0 >> 2) + j);
    if (c >= 0 && c < (n + kBlk - 1) / kBlk) return true;
  }
  return false;
}

// convolution + silu of channel c for the rows of a block (m: its first row, t: that row inside its sequence).
// TAPS: the number of taps when known at compile time (every input and weight is then loaded at once), else 0.
template <int TAPS>
__device__ __forceinline__ void conv_silu4(const DeltaParams& p, const float* hist, int c, int col, int m, int t, int pos, int C, int rows,
                                           float (&y)[kBlk]) {
  float acc[kBlk] = {};
  const float* cw = p.conv_w + static_cast<size_t>(c) * p.taps;
  if constexpr (TAPS > 0) {
    float x[TAPS + kBlk - 1], w[TAPS];
#pragma unroll
    for (int i = 0; i < TAPS; ++i) w[i] = cw[i];
#pragma unroll
    for (int i = 0; i < TAPS + kBlk - 1; ++i) {                     // input row m - (TAPS - 1) + i
      const int back = TAPS - 1 - i;
      x[i] = 0.f;
      if (-back < rows) {
        if (back <= t) x[i] = p.x[static_cast<size_t>(m - back) * p.ldx + col];
        else if (back <= pos) x[i] = hist[static_cast<size_t>((pos - back) % TAPS) * C + c];
      }
    }
#pragma unroll
    for (int r = 0; r < kBlk; ++r)
#pragma unroll
      for (int i = 0; i < TAPS; ++i) acc[r] = fmaf(x[r + i], w[i], acc[r]);
  } else {
    for (int back = p.taps - 1; back > -kBlk; --back) {             // input row m - back feeds rows r >= -back
      if (-back >= rows) break;
      float x = 0.f;
      if (back <= t) x = p.x[static_cast<size_t>(m - back) * p.ldx + col];
      else if (back <= pos) x = hist[static_cast<size_t>((pos - back) % p.taps) * C + c];
#pragma unroll
      for (int r = 0; r < kBlk; ++r) {
        const int i = p.taps - 1 - (r + back);                      // tap of this input for row r
        if (i >= 0 && i < p.taps) acc[r] = fmaf(x, cw[i], acc[r]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < kBlk; ++r) y[r] = r < rows ? silu_f32(acc[r]) : 0.f;
}


// grid (blocks, ceil((HK + H) / 4)), 128 threads; a warp per item: key heads (q, k and their dot products), value heads
template <int NI, int TAPS>
__global__ void __launch_bounds__(128) delta_prep_kernel(const __grid_constant__ DeltaParams p) {
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int item = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (item >= p.HK + p.H) return;
  int j, blk;
  if (!block_of_slot(p, blockIdx.x, j, blk)) return;
  const int slot = delta_slot(p, j);
  if (slot < 0) return;
  constexpr int DP = NI * 32;
  const int t = blk * kBlk, m = p.cu_rows[j] + t, rows = min(kBlk, p.cu_rows[j + 1] - m), pos = p.pos[m];
  const int C = 2 * p.HK * p.D + p.H * p.V;
  const float* hist = p.hist + static_cast<size_t>(slot) * p.taps * C;
  if (item < p.HK) {
    const int h = item;
    float qv[NI][kBlk], kv[NI][kBlk], sq[2][kBlk] = {};
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = i * 32 + lane;
#pragma unroll
      for (int r = 0; r < kBlk; ++r) qv[i][r] = kv[i][r] = 0.f;
      if (d < p.D) {
        conv_silu4<TAPS>(p, hist, h * p.D + d, p.q_off + h * p.D + d, m, t, pos, C, rows, qv[i]);
        conv_silu4<TAPS>(p, hist, (p.HK + h) * p.D + d, p.k_off + h * p.D + d, m, t, pos, C, rows, kv[i]);
      }
#pragma unroll
      for (int r = 0; r < kBlk; ++r) {
        sq[0][r] += qv[i][r] * qv[i][r];
        sq[1][r] += kv[i][r] * kv[i][r];
      }
    }
    float* o = p.kq + (static_cast<size_t>(blockIdx.x) * p.HK + h) * kq_words(DP);
#pragma unroll
    for (int r = 0; r < kBlk; ++r) {
      const float a = 1.f / sqrtf(warp_sum_f(sq[0][r]) + p.unit_eps) * p.q_scale;
      const float b = 1.f / sqrtf(warp_sum_f(sq[1][r]) + p.unit_eps);
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        qv[i][r] *= a;
        kv[i][r] *= b;
        o[r * DP + i * 32 + lane] = kv[i][r];
        o[(kBlk + r) * DP + i * 32 + lane] = qv[i][r];
      }
    }
    float mine = 0.f;                              // lane n keeps dot product n
#pragma unroll
    for (int i = 0; i < kBlk; ++i)
#pragma unroll
      for (int jj = 0; jj <= i; ++jj) {
        float kk = 0.f, kq = 0.f;
#pragma unroll
        for (int n = 0; n < NI; ++n) {
          if (jj < i) kk = fmaf(kv[n][jj], kv[n][i], kk);
          kq = fmaf(kv[n][jj], qv[n][i], kq);
        }
        kq = warp_sum_f(kq);
        if (lane == kq_at(i, jj)) mine = kq;
        if (jj < i) {
          kk = warp_sum_f(kk);
          if (lane == kk_at(i, jj)) mine = kk;
        }
      }
    if (lane < kPairs) o[2 * kBlk * DP + lane] = mine;
  } else {
    const int h = item - p.HK, groups = (p.VP + kCols - 1) / kCols;
    float beta = 0.f, g = 1.f;                     // lanes 0 .. 3: one token each
    if (lane < rows) {
      const float* x = p.x + static_cast<size_t>(m + lane) * p.ldx;
      beta = sigmoid_f32(x[p.b_off + h]);
      g = expf(-expf(p.A_log[h]) * softplus_f32(x[p.a_off + h] + p.dt_bias[h]));
    }
    for (int d = lane; d < groups * kCols; d += 32) {
      float y[kBlk] = {};
      if (d < p.V) conv_silu4<TAPS>(p, hist, 2 * p.HK * p.D + h * p.V + d, p.v_off + h * p.V + d, m, t, pos, C, rows, y);
      float* o = p.vb + ((static_cast<size_t>(blockIdx.x) * p.H + h) * groups + d / kCols) * kVWords + d % kCols;
#pragma unroll
      for (int r = 0; r < kBlk; ++r) o[r * kCols] = y[r];
    }
    float* o = p.vb + (static_cast<size_t>(blockIdx.x) * p.H + h) * groups * kVWords + kBlk * kCols;
    for (int gr = 0; gr < groups; ++gr)
      if (lane < kBlk) {
        o[gr * kVWords + lane] = beta;
        o[gr * kVWords + kBlk + lane] = g;
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

constexpr int kScanStages = 4;           // blocks of four tokens in flight

// grid (nseq, H, ceil(VP / 16)), 160 threads: four warps of four value columns (two lane groups of two columns, 16 lanes
// along the keys), each at its own pace, and a warp whose first lane keeps the copies going
constexpr int kScanThreads = 160;

// kCorrect = false: u_i = beta_i v_i, the rule without correction.
template <int NJ, bool kCorrect>
__global__ void __launch_bounds__(kScanThreads) delta_scan_kernel(const __grid_constant__ DeltaParams p) {
  constexpr int DP = NJ * 64;
  constexpr int kKq = kq_words(DP);
  constexpr int kStageWords = kKq + kVWords;
  extern __shared__ float4 sm4[];
  float* sm = reinterpret_cast<float*>(sm4);
  __shared__ uint64_t bars[2 * kScanStages];
  pdl_wait();
  const int j = blockIdx.x, h = blockIdx.y;
  const int r0 = p.cu_rows[j], n = p.cu_rows[j + 1] - r0;
  if (n <= 0) return;
  const int slot = delta_slot(p, j);
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 15;
  const int vb = blockIdx.z * kCols, groups = (p.VP + kCols - 1) / kCols;
  const int hk = h / (p.H / p.HK);
  const int cl = warp * 4 + (lane >> 4) * 2;       // column inside the CTA's 16
  const bool on = vb + warp * 4 < p.VP;            // VP is a multiple of 8
  const int blocks = (n + kBlk - 1) / kBlk;
  const uint32_t bar = smem_u32(bars), bar_free = bar + 8 * kScanStages;
  const uint32_t sm_u = smem_u32(sm);
  if (threadIdx.x == 0) {
    for (int i = 0; i < kScanStages; ++i) {
      mbar_init(bar + 8 * i, 1);
      mbar_init(bar_free + 8 * i, 4);
    }
    mbar_init_fence();
  }
  __syncthreads();
  if (warp == 4) {                                 // ---- copies
    if (lane == 0) {
      const size_t bs0 = static_cast<size_t>(block_slot(r0, j, 0));
      const float* kq = p.kq + (bs0 * p.HK + hk) * kKq;
      const float* vr = p.vb + ((bs0 * p.H + h) * groups + blockIdx.z) * kVWords;
      const size_t kq_step = static_cast<size_t>(p.HK) * kKq, v_step = static_cast<size_t>(p.H) * groups * kVWords;
      int blk = 0;
      for (; blk < blocks; ++blk) {
        const int s = blk % kScanStages;
        if (blk >= kScanStages && !mbar_wait(bar_free + 8 * s, ((blk / kScanStages) & 1) ^ 1, p.err, kErrWaitEmpty)) break;
        mbar_arrive_expect_tx(bar + 8 * s, kStageWords * 4);
        bulk_g2s(sm_u + s * kStageWords * 4, kq + blk * kq_step, kKq * 4, bar + 8 * s);
        bulk_g2s(sm_u + (s * kStageWords + kKq) * 4, vr + blk * v_step, kVWords * 4, bar + 8 * s);
      }
      for (int i = max(0, blk - kScanStages); i < blk; ++i)        // the CTA does not leave before its copies have landed
        mbar_wait(bar + 8 * (i % kScanStages), (i / kScanStages) & 1, p.err, kErrWaitDrain);
    }
    return;
  }
  f32x2 S[NJ][2][2] = {};                          // [64 keys][pair of keys][column]
  float* st = p.state + ((static_cast<size_t>(slot) * p.H + h) * p.VP + vb + cl) * DP;
  if (on) {
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
      for (int i = 0; i < NJ; ++i) {
        const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(st + static_cast<size_t>(c) * DP + i * 64 + lg * 4);
        S[i][0][c] = f.x;
        S[i][1][c] = f.y;
      }
  }
  const int tok = lg >> 2, col = (lg >> 1) & 1;    // whose read-out value this lane keeps (lanes 2i, 2i + 1 share one)
  float* out = p.o + (static_cast<size_t>(r0 + tok) * p.H + h) * p.VP + vb + cl + col;
  const size_t out_step = static_cast<size_t>(kBlk) * p.H * p.VP;
  const float skip = !kCorrect && p.skip != nullptr ? p.skip[h] : 0.f;
  for (int blk = 0; blk < blocks; ++blk) {
    const int s = blk % kScanStages;
    if (!mbar_wait(bar + 8 * s, (blk / kScanStages) & 1, p.err, kErrWaitFull)) break;
    const float* b = sm + s * kStageWords;
    const float* vrec = b + kKq;
    if (on) {
      constexpr bool kHold = NJ <= 2;              // the keys stay in registers for the update
      f32x2 kr[kHold ? kBlk : 1][kHold ? NJ : 1][2];
      float sk[kBlk][2], sq[kBlk][2];
#pragma unroll
      for (int r = 0; r < kBlk; ++r) {
        f32x2 a[2] = {}, c[2] = {};
#pragma unroll
        for (int i = 0; i < NJ; ++i) {
          const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(b + r * DP + i * 64 + lg * 4);
          const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(b + (kBlk + r) * DP + i * 64 + lg * 4);
          if constexpr (kHold) {
            kr[r][i][0] = k4.x;
            kr[r][i][1] = k4.y;
          }
#pragma unroll
          for (int v = 0; v < 2; ++v) {
            if constexpr (kCorrect) {
              a[v] = fma_f2(S[i][0][v], k4.x, a[v]);
              a[v] = fma_f2(S[i][1][v], k4.y, a[v]);
            }
            c[v] = fma_f2(S[i][0][v], q4.x, c[v]);
            c[v] = fma_f2(S[i][1][v], q4.y, c[v]);
          }
        }
#pragma unroll
        for (int v = 0; v < 2; ++v) {
          const float2 x = unpack_f2(a[v]), y = unpack_f2(c[v]);
          sk[r][v] = x.x + x.y;
          sq[r][v] = y.x + y.y;
        }
      }
      if constexpr (kCorrect) {
#pragma unroll
        for (int o = 1; o < 16; o <<= 1)
#pragma unroll
          for (int r = 0; r < kBlk; ++r)
#pragma unroll
            for (int v = 0; v < 2; ++v) sk[r][v] += __shfl_xor_sync(0xffffffffu, sk[r][v], o);
      }
      // read-out values by halving exchange (4 + 2 + 1 + 1 shuffles)
      float mine;
      {
        float t4[4], t2[2];
        const bool b3 = (lg & 8) != 0, b2 = (lg & 4) != 0, b1 = (lg & 2) != 0;
#pragma unroll
        for (int e = 0; e < 4; ++e) {              // tokens 0, 1 stay with b3 = 0; tokens 2, 3 with b3 = 1
          const float keep = b3 ? sq[2 + (e >> 1)][e & 1] : sq[e >> 1][e & 1];
          const float give = b3 ? sq[e >> 1][e & 1] : sq[2 + (e >> 1)][e & 1];
          t4[e] = keep + __shfl_xor_sync(0xffffffffu, give, 8);
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float keep = b2 ? t4[2 + e] : t4[e], give = b2 ? t4[e] : t4[2 + e];
          t2[e] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
        }
        const float keep = b1 ? t2[1] : t2[0], give = b1 ? t2[0] : t2[1];
        mine = keep + __shfl_xor_sync(0xffffffffu, give, 2);
        mine += __shfl_xor_sync(0xffffffffu, mine, 1);
      }
      float dl[kBlk], u[kBlk][2], pr[kPairs];
#pragma unroll
      for (int e = 0; e < kPairs; e += 4) *reinterpret_cast<float4*>(pr + e) = *reinterpret_cast<const float4*>(b + 2 * kBlk * DP + e);
      const float4 be4 = *reinterpret_cast<const float4*>(vrec + kBlk * kCols), g4 = *reinterpret_cast<const float4*>(vrec + kBlk * kCols + kBlk);
      const float beta[4] = {be4.x, be4.y, be4.z, be4.w}, g[4] = {g4.x, g4.y, g4.z, g4.w};
      float G = 1.f, o = 0.f;
#pragma unroll
      for (int i = 0; i < kBlk; ++i) {
        const float2 v = *reinterpret_cast<const float2*>(vrec + i * kCols + cl);
        G *= g[i];
        float a0 = v.x, a1 = v.y;
        if constexpr (kCorrect) {
          a0 -= G * sk[i][0];
          a1 -= G * sk[i][1];
        }
#pragma unroll
        for (int jj = 0; jj < i; ++jj) {
          dl[jj] *= g[i];                          // D_ij
          if constexpr (kCorrect) {
            const float w = dl[jj] * pr[kk_at(i, jj)];
            a0 = fmaf(-w, u[jj][0], a0);
            a1 = fmaf(-w, u[jj][1], a1);
          }
        }
        dl[i] = 1.f;
        u[i][0] = beta[i] * a0;
        u[i][1] = beta[i] * a1;
        float t = G * mine;
        if constexpr (!kCorrect) t = fmaf(skip, col ? v.y : v.x, t);
#pragma unroll
        for (int jj = 0; jj <= i; ++jj) t = fmaf(dl[jj] * pr[kq_at(i, jj)], col ? u[jj][1] : u[jj][0], t);
        o = tok == i ? t : o;
      }
      if ((lg & 1) == 0 && blk * kBlk + tok < n) out[blk * out_step] = o;
      const f32x2 G2 = pack_f2(G, G);
#pragma unroll
      for (int i = 0; i < NJ; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          S[i][e][0] = mul_f2(S[i][e][0], G2);
          S[i][e][1] = mul_f2(S[i][e][1], G2);
        }
#pragma unroll
      for (int r = 0; r < kBlk; ++r) {             // D_4r is where the recurrence left it
        const float w0 = u[r][0] * dl[r], w1 = u[r][1] * dl[r];
        const f32x2 u0 = pack_f2(w0, w0), u1 = pack_f2(w1, w1);
#pragma unroll
        for (int i = 0; i < NJ; ++i) {
          f32x2 ka, kb;
          if constexpr (kHold) {
            ka = kr[r][i][0];
            kb = kr[r][i][1];
          } else {
            const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(b + r * DP + i * 64 + lg * 4);
            ka = k4.x;
            kb = k4.y;
          }
          S[i][0][0] = fma_f2(u0, ka, S[i][0][0]);
          S[i][0][1] = fma_f2(u1, ka, S[i][0][1]);
          S[i][1][0] = fma_f2(u0, kb, S[i][1][0]);
          S[i][1][1] = fma_f2(u1, kb, S[i][1][1]);
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
      for (int i = 0; i < NJ; ++i)
        *reinterpret_cast<ulonglong2*>(st + static_cast<size_t>(c) * DP + i * 64 + lg * 4) = make_ulonglong2(S[i][0][c], S[i][1][c]);
  }
}

// Gated norm of one head row (o: V values, shared or global memory) by a warp.
__device__ __forceinline__ void delta_gated_norm(const DeltaParams& p, const float* o, int m, int h, int lane) {
  float sq = 0.f;
  for (int v = lane; v < p.V; v += 32) sq += o[v] * o[v];
  const float r = 1.f / sqrtf(warp_sum_f(sq) / static_cast<float>(p.V) + p.eps);
  const float* g = p.x + static_cast<size_t>(m) * p.ldx + p.g_off + h * p.V;
  if ((p.V & 3) == 0) {                            // (the gate's columns start at a multiple of 8, VP is one too)
    for (int v = lane * 4; v < p.V; v += 128) {
      const float4 a = *reinterpret_cast<const float4*>(o + v), b = *reinterpret_cast<const float4*>(g + v),
                   w = *reinterpret_cast<const float4*>(p.norm_w + v);
      operand_store4(p.out, m, p.out_k0 + h * p.V + v,
                     make_float4(a.x * r * w.x * silu_f32(b.x), a.y * r * w.y * silu_f32(b.y), a.z * r * w.z * silu_f32(b.z),
                                 a.w * r * w.w * silu_f32(b.w)));
    }
    return;
  }
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

template <int NI, int TAPS>
static cudaError_t delta_prep(const DeltaParams& p, cudaStream_t stream) {
  return launch(delta_prep_kernel<NI, TAPS>, dim3(p.M / kBlk + p.nseq, (p.HK + p.H + 3) / 4), dim3(128), 0, stream, 0, p);
}

template <int NJ, bool kCorrect>
static int delta_scan(const DeltaParams& p, cudaStream_t stream) {
  constexpr int smem = kScanStages * (kq_words(NJ * 64) + kVWords) * 4;
  static bool ready[64];
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return static_cast<int>(cudaErrorInvalidDevice);
  if (!ready[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<NJ, kCorrect>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    ready[dev] = true;
  }
  return static_cast<int>(launch(delta_scan_kernel<NJ, kCorrect>, dim3(p.nseq, p.H, (p.VP + kCols - 1) / kCols), dim3(kScanThreads), smem,
                                 stream, 0, p));
}

template <int NJ>
static int delta_go(const DeltaParams& p, bool single, cudaStream_t stream) {
  constexpr int NI = NJ * 2;
  if (single) {
    const int warps = min(8, p.VP / 8);
    const int smem = (2 * NI * 32 + 2 * p.VP) * 4;
    return static_cast<int>(launch(delta_step_kernel<NI>, dim3(p.H, p.nseq), dim3(32 * warps), smem, stream, 0, p));
  }
  int e = static_cast<int>(p.taps == 4 ? delta_prep<NI, 4>(p, stream) : delta_prep<NI, 0>(p, stream));
  if (e == 0) e = delta_scan<NJ, true>(p, stream);
  if (e == 0) e = static_cast<int>(launch(delta_out_kernel, dim3(p.M + p.nseq, (p.H + 7) / 8), dim3(256), 0, stream, 0, p));
  return e;
}

}  // namespace saber

extern "C" int saber_delta_launches(int single_row) { return single_row ? 1 : 3; }

extern "C" int saber_delta_launch(const saber::DeltaParams* p, int single_row, cudaStream_t stream) {
  using namespace saber;
  if (p->M <= 0 || p->nseq <= 0 || p->HK <= 0 || p->H % p->HK || p->D > p->DP || (p->VP & 7) || p->V > p->VP || p->VP > 4096 || p->taps < 1)
    return static_cast<int>(cudaErrorInvalidValue);
  switch (p->DP) {
    case 64: return delta_go<1>(*p, single_row != 0, stream);
    case 128: return delta_go<2>(*p, single_row != 0, stream);
    case 192: return delta_go<3>(*p, single_row != 0, stream);
    case 256: return delta_go<4>(*p, single_row != 0, stream);
    case 384: return delta_go<6>(*p, single_row != 0, stream);
    case 512: return delta_go<8>(*p, single_row != 0, stream);
    default: return static_cast<int>(cudaErrorInvalidValue);
  }
}

int saber_outer_scan_launch(const saber::DeltaParams* p, cudaStream_t stream) {
  using namespace saber;
  switch (p->DP) {
    case 64: return delta_scan<1, false>(*p, stream);
    case 128: return delta_scan<2, false>(*p, stream);
    case 192: return delta_scan<3, false>(*p, stream);
    case 256: return delta_scan<4, false>(*p, stream);
    case 384: return delta_scan<6, false>(*p, stream);
    case 512: return delta_scan<8, false>(*p, stream);
    default: return static_cast<int>(cudaErrorInvalidValue);
  }
}
