// Decayed outer products with free head sizes, fp32 throughout.
//
// Prompt portions (ragged rows, any length): three launches.
//   prep   convolution, silu, decay and weight of every token as the records of the scan in delta.cu
//   scan   that scan without its correction term: four tokens at a time, a warp per four value columns, the state in
//          registers (fp32 models and sizes the chunk form of ssd_chunk.cu does not take)
//   out    gate and grouped norm into the operand of the output linear; the convolution inputs go to the ring
// Decoding (one row per sequence): one launch, a CTA per (head, sequence); the last CTA of a norm group to
// finish norms it.
#include "delta.h"
#include "launch.cuh"
#include "ssd_chunk.h"
#include "ssd_device.cuh"

namespace saber {

// grid (blocks, ceil((HK + H) / 4)), 128 threads; a warp per item: key heads (q, k and their dot products), value heads
template <int NI, int TAPS>
__global__ void __launch_bounds__(128) ssd_prep_kernel(const __grid_constant__ SsdParams p) {
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int item = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (item >= p.HK + p.H) return;
  int j = 0, blk = 0;
  bool found = false;
  for (; j < p.nseq; ++j) {
    const int r0 = p.cu_rows[j], n = p.cu_rows[j + 1] - r0;
    blk = static_cast<int>(blockIdx.x) - block_slot(r0, j, 0);
    if (blk >= 0 && blk < (n + kBlk - 1) / kBlk) { found = true; break; }
  }
  if (!found) return;
  const int slot = ssd_slot(p, j);
  if (slot < 0) return;
  constexpr int DP = NI * 32;
  const int t = blk * kBlk, m = p.cu_rows[j] + t, rows = min(kBlk, p.cu_rows[j + 1] - m), pos = p.pos[m];
  const int C = ssd_channels(p);
  const float* hist = p.hist + static_cast<size_t>(slot) * p.taps * C;
  if (item < p.HK) {
    const int h = item;
    float qv[NI][kBlk], kv[NI][kBlk];
    float* o = p.kq + (static_cast<size_t>(blockIdx.x) * p.HK + h) * kq_words(DP);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = i * 32 + lane;
#pragma unroll
      for (int r = 0; r < kBlk; ++r) qv[i][r] = kv[i][r] = 0.f;
      if (d < p.N) {
        ssd_inputs<kBlk, TAPS>(p, hist, h * p.N + d, m, t, pos, C, rows, qv[i]);
        ssd_inputs<kBlk, TAPS>(p, hist, (p.HK + h) * p.N + d, m, t, pos, C, rows, kv[i]);
      }
#pragma unroll
      for (int r = 0; r < kBlk; ++r) {
        o[r * DP + d] = kv[i][r];
        o[(kBlk + r) * DP + d] = qv[i][r];
      }
    }
    float mine = 0.f;                              // lane n keeps dot product n
#pragma unroll
    for (int i = 0; i < kBlk; ++i)
#pragma unroll
      for (int jj = 0; jj <= i; ++jj) {
        float kq = 0.f;
#pragma unroll
        for (int n = 0; n < NI; ++n) kq = fmaf(kv[n][jj], qv[n][i], kq);
        kq = warp_sum_f(kq);
        if (lane == kq_at(i, jj)) mine = kq;
      }
    if (lane < kPairs) o[2 * kBlk * DP + lane] = mine;
  } else {
    const int h = item - p.HK, groups = (p.VP + kCols - 1) / kCols;
    float w = 0.f, a = 1.f, la;                    // lanes 0 .. 3: one token each
    if (lane < rows) ssd_gates(p, m + lane, h, a, w, la);
    for (int d = lane; d < groups * kCols; d += 32) {
      float y[kBlk] = {};
      if (d < p.V) ssd_inputs<kBlk, TAPS>(p, hist, 2 * p.HK * p.N + h * p.V + d, m, t, pos, C, rows, y);
      float* o = p.vb + ((static_cast<size_t>(blockIdx.x) * p.H + h) * groups + d / kCols) * kVWords + d % kCols;
#pragma unroll
      for (int r = 0; r < kBlk; ++r) o[r * kCols] = y[r];
    }
    float* o = p.vb + (static_cast<size_t>(blockIdx.x) * p.H + h) * groups * kVWords + kBlk * kCols;
    for (int gr = 0; gr < groups; ++gr)
      if (lane < kBlk) {
        o[gr * kVWords + lane] = w;
        o[gr * kVWords + kBlk + lane] = a;
      }
  }
}

// Sum over the threads of a block (nw warps); red: nw floats of shared memory.
__device__ __forceinline__ float block_sum(float v, float* red, int nw) {
  v = warp_sum_f(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = 0.f;
  for (int w = 0; w < nw; ++w) v += red[w];
  return v;
}

struct Silu { __device__ __forceinline__ float operator()(float x) const { return silu_f32(x); } };
struct Sigmoid { __device__ __forceinline__ float operator()(float x) const { return sigmoid_f32(x); } };
// v times f(g) where it applies
template <typename Fn>
__device__ __forceinline__ float4 gate4(bool on, float4 v, float4 g, Fn f) {
  if (!on) return v;
  return make_float4(v.x * f(g.x), v.y * f(g.y), v.z * f(g.z), v.w * f(g.w));
}
__device__ __forceinline__ float square4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// Gate and norm of one group of a row (o: the row's read-outs [H][VP], n values of the group) by a block.
__device__ __forceinline__ void ssd_gated_norm(const SsdParams& p, const float* o, int m, int grp, int n, float* red) {
  const int nt = blockDim.x, c0 = grp * n, k0 = p.out_k0 + c0;
  const float* g = p.x + static_cast<size_t>(m) * p.ldx + p.g_off + c0;
  const float* w = p.norm_w + c0;
  const bool first = p.gate_first != 0;
  if (((p.V | n) & 3) == 0) {                      // sixteen values a thread at a time, held where that is all
    constexpr int kHeld = 4;
    float4 v[kHeld], gate[kHeld];
    auto load = [&](int base) {
#pragma unroll
      for (int u = 0; u < kHeld; ++u) {
        const int i = base + (u * nt + threadIdx.x) * 4, c = c0 + i, h = c / p.V;
        v[u] = gate[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < n) {
          v[u] = __ldcg(reinterpret_cast<const float4*>(o + h * p.VP + c - h * p.V));
          gate[u] = *reinterpret_cast<const float4*>(g + i);
        }
      }
#pragma unroll
      for (int u = 0; u < kHeld; ++u) v[u] = gate4(first, v[u], gate[u], Silu{});
    };
    const int span = 4 * kHeld * nt;
    float sq = 0.f;
    for (int base = 0; base < n; base += span) {
      load(base);
#pragma unroll
      for (int u = 0; u < kHeld; ++u) sq += square4(v[u]);
    }
    const float r = 1.f / sqrtf(block_sum(sq, red, nt >> 5) / static_cast<float>(n) + p.eps);
    for (int base = 0; base < n; base += span) {
      if (n > span) load(base);
#pragma unroll
      for (int u = 0; u < kHeld; ++u) {
        const int i = base + (u * nt + threadIdx.x) * 4;
        if (i >= n) break;
        const float4 wt = *reinterpret_cast<const float4*>(w + i);
        operand_store4(p.out, m, k0 + i,
                       gate4(!first, make_float4(v[u].x * r * wt.x, v[u].y * r * wt.y, v[u].z * r * wt.z, v[u].w * r * wt.w), gate[u], Sigmoid{}));
      }
    }
    return;
  }
  auto gated = [&](int i) {
    const int c = c0 + i, h = c / p.V;
    const float v = __ldcg(o + h * p.VP + c - h * p.V);
    return first ? v * silu_f32(g[i]) : v;
  };
  float sq = 0.f;
  for (int i = threadIdx.x; i < n; i += nt) {
    const float v = gated(i);
    sq += v * v;
  }
  const float r = 1.f / sqrtf(block_sum(sq, red, nt >> 5) / static_cast<float>(n) + p.eps);
  for (int i = threadIdx.x; i < n; i += nt) {
    const float y = gated(i) * r * w[i];
    operand_store1(p.out, m, k0 + i, first ? y : y * sigmoid_f32(g[i]));
  }
}

// The same by a warp, for groups of up to 1024 values.
__device__ __forceinline__ void ssd_gated_norm_warp(const SsdParams& p, const float* o, int m, int grp, int n, int lane) {
  const int c0 = grp * n, k0 = p.out_k0 + c0;
  const float* g = p.x + static_cast<size_t>(m) * p.ldx + p.g_off + c0;
  float4 v[8], gate[8];
#pragma unroll
  for (int u = 0; u < 8; ++u) {
    const int i = (u * 32 + lane) * 4, c = c0 + i, h = c / p.V;
    v[u] = gate[u] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < n) {
      v[u] = *reinterpret_cast<const float4*>(o + h * p.VP + c - h * p.V);
      gate[u] = *reinterpret_cast<const float4*>(g + i);
    }
  }
  const bool first = p.gate_first != 0;
  float sq = 0.f;
#pragma unroll
  for (int u = 0; u < 8; ++u) {
    v[u] = gate4(first, v[u], gate[u], Silu{});
    sq += square4(v[u]);
  }
  const float r = 1.f / sqrtf(warp_sum_f(sq) / static_cast<float>(n) + p.eps);
#pragma unroll
  for (int u = 0; u < 8; ++u) {
    const int i = (u * 32 + lane) * 4;
    if (i >= n) break;
    const float4 wt = *reinterpret_cast<const float4*>(p.norm_w + c0 + i);
    operand_store4(p.out, m, k0 + i,
                   gate4(!first, make_float4(v[u].x * r * wt.x, v[u].y * r * wt.y, v[u].z * r * wt.z, v[u].w * r * wt.w), gate[u], Sigmoid{}));
  }
}

// Items 0 .. items - 1 of the grid norm the rows: a warp per (row, group) (small = 1) or a CTA (small = 0); the last
// nseq * kRingBlocks CTAs update the rings.  256 threads.
constexpr int kRingBlocks = 8;

__global__ void __launch_bounds__(256, 3) ssd_out_kernel(const __grid_constant__ SsdParams p, const int items, const int small) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const int n = p.H * p.V / p.groups;
  if (static_cast<int>(blockIdx.x) < items) {
    const int item = small ? blockIdx.x * 8 + (threadIdx.x >> 5) : blockIdx.x;
    const int m = item / p.groups, g = item - m * p.groups;
    if (m >= p.M || seq_of_row(p.cu_rows, p.nseq, m) < 0) return;
    const float* o = p.o + static_cast<size_t>(m) * p.H * p.VP;
    if (small)
      ssd_gated_norm_warp(p, o, m, g, n, threadIdx.x & 31);
    else
      ssd_gated_norm(p, o, m, g, n, red);
    return;
  }
  if (p.taps == 0) return;
  const int rb = blockIdx.x - items, j = rb / kRingBlocks;
  const int r0 = p.cu_rows[j], rows = p.cu_rows[j + 1] - r0;
  const int slot = rows > 0 ? ssd_slot(p, j) : -1;
  if (slot < 0) return;
  const int C = ssd_channels(p);
  float* hist = p.hist + static_cast<size_t>(slot) * p.taps * C;
  for (int c = (rb % kRingBlocks) * 256 + threadIdx.x; c < C; c += kRingBlocks * 256) {
    const int col = ssd_column(p, c);
    for (int t = max(0, rows - p.taps); t < rows; ++t) {
      const int m = r0 + t;
      hist[static_cast<size_t>(p.pos[m] % p.taps) * C + c] = p.x[static_cast<size_t>(m) * p.ldx + col];
    }
  }
}

// One row per sequence: grid (H, nseq), 32 * min(8, VP / 8) threads.  A warp owns eight value columns at a time, eight
// lanes along the keys and two columns each.
template <int NI, int TAPS>
__global__ void __launch_bounds__(256) ssd_step_kernel(const __grid_constant__ SsdParams p) {
  extern __shared__ float4 sm4[];
  constexpr int DP = NI * 32;
  float* ks = reinterpret_cast<float*>(sm4);       // DP
  float* qs = ks + DP;                             // DP
  float* vs = qs + DP;                             // VP
  __shared__ float red[8];
  __shared__ uint32_t last_s;
  const int h = blockIdx.x, j = blockIdx.y;
  const int m = p.cu_rows[j];
  if (p.cu_rows[j + 1] <= m) return;
  const int slot = ssd_slot(p, j);
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 7, nt = blockDim.x, nw = nt >> 5;
  const size_t st0 = (static_cast<size_t>(slot) * p.H + h) * p.VP;
  const int cl = (lane >> 3) * 2;
  float4 S[2][NI];                                 // [column][32 keys]
  auto state_at = [&](int cb, int c, int i) { return reinterpret_cast<float4*>(p.state + (st0 + cb + cl + c) * DP + i * 32 + lg * 4); };
  auto load = [&](int cb) {
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
      for (int i = 0; i < NI; ++i) S[c][i] = *state_at(cb, c, i);
  };
  // the state is requested ahead of the wait: the index tables and this layer's state were complete before the step began
  // (the block has VP / 8 warps at most)
  load(warp * 8);
  pdl_trigger();                                   // the output linear fetches its first weights beside the last CTAs of this grid
  pdl_wait();
  const int pos = p.pos[m], share = p.H / p.HK, hk = h / share;
  const int C = ssd_channels(p);
  float* hist = p.hist + static_cast<size_t>(slot) * p.taps * C;
  const float* x = p.x + static_cast<size_t>(m) * p.ldx;
  float a, w, la;
  ssd_gates(p, m, h, a, w, la);
  const size_t now = p.taps ? static_cast<size_t>(pos % p.taps) * C : 0;
  for (int d = threadIdx.x; d < 2 * DP; d += nt) {
    const int isk = d >= DP ? 1 : 0, n = d - isk * DP;
    float y[1] = {0.f};
    if (n < p.N) {
      const int c = (isk * p.HK + hk) * p.N + n;
      ssd_inputs<1, TAPS>(p, hist, c, m, 0, pos, C, 1, y);
      if (p.taps && h % share == 0) hist[now + c] = x[ssd_column(p, c)];      // ring row of this token: no head of this step reads it
    }
    (isk ? ks : qs)[n] = y[0];
  }
  for (int d = threadIdx.x; d < p.VP; d += nt) {
    float y[1] = {0.f};
    if (d < p.V) {
      const int c = 2 * p.HK * p.N + h * p.V + d;
      ssd_inputs<1, TAPS>(p, hist, c, m, 0, pos, C, 1, y);
      if (p.taps) hist[now + c] = x[ssd_column(p, c)];
    }
    vs[d] = y[0];
  }
  __syncthreads();
  const float skip = p.skip ? p.skip[h] : 0.f;
  float* row = p.o + static_cast<size_t>(m) * p.H * p.VP + h * p.VP;
  for (int cb = warp * 8; cb < p.VP; cb += nw * 8) {
    if (cb != warp * 8) load(cb);
    const float u[2] = {w * vs[cb + cl], w * vs[cb + cl + 1]};
    float o[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const float4 k = *reinterpret_cast<const float4*>(ks + i * 32 + lg * 4), q = *reinterpret_cast<const float4*>(qs + i * 32 + lg * 4);
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        float4& s = S[c][i];
        s.x = fmaf(u[c], k.x, a * s.x);
        s.y = fmaf(u[c], k.y, a * s.y);
        s.z = fmaf(u[c], k.z, a * s.z);
        s.w = fmaf(u[c], k.w, a * s.w);
        o[c] = fmaf(s.x, q.x, o[c]);
        o[c] = fmaf(s.y, q.y, o[c]);
        o[c] = fmaf(s.z, q.z, o[c]);
        o[c] = fmaf(s.w, q.w, o[c]);
        *state_at(cb, c, i) = s;
      }
    }
#pragma unroll
    for (int s = 1; s < 8; s <<= 1) {
      o[0] += __shfl_xor_sync(0xffffffffu, o[0], s);
      o[1] += __shfl_xor_sync(0xffffffffu, o[1], s);
    }
    if (lg < 2) __stcg(row + cb + cl + lg, fmaf(skip, vs[cb + cl + lg], lg ? o[1] : o[0]));
  }
  // the last head to arrive norms the row, or the norm group where groups hold whole heads
  const int parts = p.H % p.groups == 0 ? p.groups : 1, per = p.H / parts, part = h / per;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    uint32_t* cnt = p.counters + j * parts + part;
    const bool last = atomicAdd(cnt, 1u) == static_cast<uint32_t>(per) - 1u;
    if (last) *cnt = 0u;
    __threadfence();
    last_s = last ? 1u : 0u;
  }
  __syncthreads();
  if (!last_s) return;
  for (int g = part; g < p.groups; g += parts)
    ssd_gated_norm(p, p.o + static_cast<size_t>(m) * p.H * p.VP, m, g, p.H * p.V / p.groups, red);
}

template <int NI>
static cudaError_t ssd_step(const SsdParams& p, cudaStream_t stream) {
  const dim3 grid(p.H, p.nseq), block(32 * (p.VP / 8 < 8 ? p.VP / 8 : 8));
  const int smem = (2 * NI * 32 + p.VP) * 4;
  return p.taps == 4   ? launch(ssd_step_kernel<NI, 4>, grid, block, smem, stream, 2, p)
         : p.taps == 0 ? launch(ssd_step_kernel<NI, -1>, grid, block, smem, stream, 2, p)
                       : launch(ssd_step_kernel<NI, 0>, grid, block, smem, stream, 2, p);
}
template <int NI>
static cudaError_t ssd_prep(const SsdParams& p, cudaStream_t stream) {
  const dim3 grid(p.M / kBlk + p.nseq, (p.HK + p.H + 3) / 4);
  return p.taps == 0 ? launch(ssd_prep_kernel<NI, -1>, grid, dim3(128), 0, stream, 0, p)
                     : launch(ssd_prep_kernel<NI, 0>, grid, dim3(128), 0, stream, 0, p);
}

template <int NI>
static int ssd_go(const SsdParams& p, bool single, cudaStream_t stream) {
  if (single) return static_cast<int>(ssd_step<NI>(p, stream));
  int e = static_cast<int>(ssd_prep<NI>(p, stream));
  if (e == 0) {
    DeltaParams d = {};
    d.state = p.state;
    d.kq = p.kq;
    d.vb = p.vb;
    d.o = p.o;
    d.cu_rows = p.cu_rows;
    d.slots = p.slots;
    d.nseq = p.nseq;
    d.H = p.H;
    d.HK = p.HK;
    d.DP = p.DP;
    d.VP = p.VP;
    d.n_slots = p.n_slots;
    d.skip = p.skip;
    d.err = p.err;
    e = saber_outer_scan_launch(&d, stream);
  }
  return e;
}

}  // namespace saber

extern "C" int saber_ssd_launches(const saber::SsdParams* p, int single_row) { return single_row ? 1 : 1 + (p->chunk ? saber_ssd_chunk_launches() : 2); }

extern "C" int saber_ssd_launch(const saber::SsdParams* p, int single_row, cudaStream_t stream) {
  using namespace saber;
  if (p->M <= 0 || p->nseq <= 0 || p->HK <= 0 || p->H % p->HK || p->N > p->DP || (p->VP & 7) || p->V > p->VP || p->VP > 4096 || p->taps < 0 ||
      p->groups <= 0 || (p->H * p->V) % p->groups ||
      (p->dt_off < 0 ? p->decay == nullptr : (p->A_log == nullptr || p->dt_bias == nullptr)) || (p->taps > 0 && (p->conv_w == nullptr || p->hist == nullptr)) ||
      p->o == nullptr || p->state == nullptr || (single_row ? p->counters == nullptr : (p->chunk == nullptr && (p->kq == nullptr || p->vb == nullptr))))
    return static_cast<int>(cudaErrorInvalidValue);
  int e;
  if (!single_row && p->chunk) {
    e = saber_ssd_chunk_launch(p, stream);
  } else {
    switch (p->DP) {
      case 64: e = ssd_go<2>(*p, single_row != 0, stream); break;
      case 128: e = ssd_go<4>(*p, single_row != 0, stream); break;
      case 192: e = ssd_go<6>(*p, single_row != 0, stream); break;
      case 256: e = ssd_go<8>(*p, single_row != 0, stream); break;
      case 384: e = ssd_go<12>(*p, single_row != 0, stream); break;
      case 512: e = ssd_go<16>(*p, single_row != 0, stream); break;
      default: return static_cast<int>(cudaErrorInvalidValue);
    }
  }
  if (e != 0 || single_row) return e;
  const int n = p->H * p->V / p->groups, small = n <= 1024 && ((p->V | n) & 3) == 0 ? 1 : 0;
  const int items = small ? (p->M * p->groups + 7) / 8 : p->M * p->groups;
  return static_cast<int>(launch(ssd_out_kernel, dim3(items + p->nseq * kRingBlocks), dim3(256), 0, stream, 0, *p, items, small));
}
