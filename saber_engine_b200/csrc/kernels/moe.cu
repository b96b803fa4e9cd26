// Mixture-of-experts routing for sm_100a: softmax over the router logits, top-k (lower id wins
// ties), optional renormalisation, then an expert-major placement of the routes into 16-row-padded
// segments plus the tile table the grouped GEMM walks, and the weighted combine.
//
// Parity: crates/saber-kernels/hip/moe_route.hip:1-30 (softmax fp32 -> top-10, lower id wins ties ->
// renorm -> expert-major sort into 16-row blocks + tile tables; only this rank's experts are placed)
// and moe_combine_bf16 (sum of w * Y in top-k order + shared expert).  Three launches here:
// topk (warp per token), plan (one block: scan, tile table), place (thread per route).
#include "launch.cuh"
#include "moe.h"
#include "gemm_i8.h"
#include <math.h>
#include <cuda_fp8.h>

namespace saber {

constexpr int kMoeTpMaxTiles = kTpMaxTiles;   // same flag regions as the row-parallel GEMM

__device__ __forceinline__ float e_safe(float x, float mx) { return x == -INFINITY ? 0.f : __expf(x - mx); }

__device__ __forceinline__ float moe_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// Routes by sigmoid scores with a correction of the choice (MoeRouteParams::sigmoid).
template <int kPer, typename Add>
__device__ __forceinline__ void moe_sigmoid_row(const MoeRouteParams& p, int m, int lane, const Add& add) {
  const float* z = p.logits_f32 + static_cast<size_t>(m) * p.ld;
  float v[kPer];                                    // choice scores (they may be negative)
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    const int e = i * 32 + lane;
    v[i] = e < p.E ? moe_sigmoid(z[e]) + (p.correction != nullptr ? p.correction[e] : 0.f) : -INFINITY;
  }
  // largest of the values with their bit in `among`, entry i * 32 + lane below n; the lower entry wins ties (n: none is a number)
  auto best = [&](const float (&x)[kPer], uint32_t among, int n, float& bv, int& be) {
    bv = -INFINITY;
    be = n;
#pragma unroll
    for (int i = 0; i < kPer; ++i)
      if ((among >> i & 1u) && i * 32 + lane < n && x[i] > bv) { bv = x[i]; be = i * 32 + lane; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ov > bv || (ov == bv && oe < be)) { bv = ov; be = oe; }
    }
  };
  const uint32_t all = kPer == 32 ? 0xffffffffu : (1u << (kPer & 31)) - 1u;
  uint32_t open = all;
  if (p.groups > 1 && p.keep < p.groups) {
    const int size = p.E / p.groups;
    float strength[kPer];                           // entry i * 32 + lane: a group
#pragma unroll
    for (int i = 0; i < kPer; ++i) strength[i] = -INFINITY;
    for (int g = 0; g < p.groups; ++g) {
      uint32_t in = 0u;
#pragma unroll
      for (int i = 0; i < kPer; ++i) {
        const int e = i * 32 + lane;
        if (e >= g * size && e < (g + 1) * size) in |= 1u << i;
      }
      float a, b = 0.f;
      int ea, eb;
      best(v, in, p.E, a, ea);
      if (size > 1) {
        if ((ea & 31) == lane) in &= ~(1u << (ea >> 5 & 31));
        best(v, in, p.E, b, eb);
      }
#pragma unroll
      for (int i = 0; i < kPer; ++i)
        if (i * 32 + lane == g) strength[i] = a + b;
    }
    uint32_t left = all;
    open = 0u;
    for (int k = 0; k < p.keep; ++k) {
      float bv;
      int g;
      best(strength, left, p.groups, bv, g);
      if (g >= p.groups) break;                     // (scores that are no numbers)
      if ((g & 31) == lane) left &= ~(1u << (g >> 5));
#pragma unroll
      for (int i = 0; i < kPer; ++i) {
        const int e = i * 32 + lane;
        if (e >= g * size && e < (g + 1) * size) open |= 1u << i;
      }
    }
  }
  float sum = 0.f, mine_w = 0.f;
  int mine_e = -1;                                  // lane k holds route k
  for (int k = 0; k < p.top_k; ++k) {
    float bv;
    int be;
    best(v, open, p.E, bv, be);
    if (be >= p.E) break;
    if ((be & 31) == lane) open &= ~(1u << (be >> 5));
    const float s = moe_sigmoid(z[be]);             // (the score itself; the choice's had the correction)
    sum += s;
    if (lane == k) { mine_w = s; mine_e = be; }
  }
  if (lane < p.top_k) {
    p.topk_id[m * p.top_k + lane] = mine_e;
    p.topk_w[m * p.top_k + lane] = mine_w / (sum + 1e-20f) * p.scale;
    const int le = mine_e - p.e_lo;
    if (mine_e >= 0 && le >= 0 && le < p.e_n) add(le);
  }
}

// The routes of token m, by one warp; kPer * 32 experts at most.  add(expert) counts a route of a local expert.
template <int kPer, bool kSigmoid, typename Add>
__device__ __forceinline__ void moe_topk_row(const MoeRouteParams& p, int m, int lane, const Add& add) {
  if (p.live != nullptr && m >= *p.live) {
    for (int k = lane; k < p.top_k; k += 32) {
      p.topk_id[m * p.top_k + k] = -1;
      p.topk_w[m * p.top_k + k] = 0.f;
    }
    return;
  }
  if constexpr (kSigmoid) {
    moe_sigmoid_row<kPer>(p, m, lane, add);
    return;
  }
  float v[kPer];
  float mx = -INFINITY;
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    const int e = i * 32 + lane;
    const size_t at = static_cast<size_t>(m) * p.ld + e;
    v[i] = e >= p.E ? -INFINITY : p.logits_f32 != nullptr ? p.logits_f32[at] : __bfloat162float(p.logits[at]);
    mx = fmaxf(mx, v[i]);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    v[i] = v[i] == -INFINITY ? 0.f : p.logits_f32 != nullptr ? expf(v[i] - mx) : e_safe(v[i], mx);
    sum += v[i];
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  uint32_t open = kPer == 32 ? 0xffffffffu : (1u << kPer) - 1u;     // bit i: expert i * 32 + lane may be chosen
  auto best = [&](uint32_t among, float& bv, int& be) {             // largest score, the lower id wins ties
    bv = -1.f;
    be = p.E;
#pragma unroll
    for (int i = 0; i < kPer; ++i)
      if ((among >> i & 1u) && i * 32 + lane < p.E && v[i] > bv) { bv = v[i]; be = i * 32 + lane; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ov > bv || (ov == bv && oe < be)) { bv = ov; be = oe; }
    }
  };
  if (p.groups > 1 && p.keep < p.groups) {
    // the best expert outside the groups kept so far names the next group to keep
    const int size = p.E / p.groups;
    uint32_t kept = 0u;
    for (int k = 0; k < p.keep; ++k) {
      float bv;
      int be;
      best(~kept, bv, be);
      if (be >= p.E) break;                         // (scores that are no numbers)
      const int lo = be / size * size;
#pragma unroll
      for (int i = 0; i < kPer; ++i) {
        const int e = i * 32 + lane;
        if (e >= lo && e < lo + size) kept |= 1u << i;
      }
    }
    open = kept;
  }
  float wsum = 0.f, mine_w = 0.f;
  int mine_e = -1;                                  // lane k holds route k
  for (int k = 0; k < p.top_k; ++k) {
    float bv;
    int be;
    best(open, bv, be);
    if (be >= p.E) break;
    wsum += bv;
    if (lane == k) { mine_w = bv; mine_e = be; }
    if ((be & 31) == lane) open &= ~(1u << (be >> 5));
  }
  if (lane < p.top_k) {
    p.topk_id[m * p.top_k + lane] = mine_e;
    p.topk_w[m * p.top_k + lane] = mine_w / (p.norm_topk ? wsum : sum);
    const int le = mine_e - p.e_lo;
    if (mine_e >= 0 && le >= 0 && le < p.e_n) add(le);
  }
}

// grid = ceil(M / 8), block 256: one warp per token.
template <int kPer, bool kSigmoid>
__global__ void __launch_bounds__(256) moe_topk_kernel(const MoeRouteParams p) {
  pdl_wait();
  const int m = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (m < p.M) moe_topk_row<kPer, kSigmoid>(p, m, threadIdx.x & 31, [&](int e) { atomicAdd(p.counts + e, 1); });
}

// One block of 1024 threads (one per local expert): exclusive scans of the padded row counts and of
// the tile counts (warp shuffles, then the 32 warp totals), every thread writes its expert's tiles;
// cursors and counts are cleared for the placement pass and for the next step's routing.
__device__ __forceinline__ int block_excl_scan_1024(int v, int* warp_tot, int& total) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
  int inc = v;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int n = __shfl_up_sync(0xffffffffu, inc, o);
    if (lane >= o) inc += n;
  }
  __syncthreads();                       // warp_tot may still be read by the previous scan
  if (lane == 31) warp_tot[w] = inc;
  __syncthreads();
  int base = 0, tot = 0;
#pragma unroll
  for (int k = 0; k < 32; ++k) {
    const int x = warp_tot[k];
    if (k < w) base += x;
    tot += x;
  }
  total = tot;
  return base + inc - v;
}

__global__ void __launch_bounds__(1024) moe_plan_kernel(const MoeRouteParams p) {
  pdl_wait();
  __shared__ int warp_tot[32];
  const int t = threadIdx.x;
  int c = 0;
  if (t < p.e_n) {
    c = p.counts[t];
    p.counts[t] = 0;                     // the next routing pass accumulates from zero
    p.cursors[t] = 0;
  }
  int rows_total, tiles_total;
  const int off = block_excl_scan_1024((c + 15) & ~15, warp_tot, rows_total);
  const int toff = block_excl_scan_1024((c + p.nt - 1) / p.nt, warp_tot, tiles_total);
  if (t < p.e_n) {
    p.offsets[t] = off;
    int i = toff;
    for (int r = 0; r < c; r += p.nt) p.tiles[i++] = make_int4(t, off + r, min(p.nt, c - r), 0);
  }
  if (t == 0) {
    p.offsets[p.e_n] = rows_total;
    p.ntiles[0] = tiles_total;
    p.ntiles[1] = rows_total;
  }
  for (int i = t; i < p.rows_cap; i += blockDim.x) p.src_row[i] = -1;
}

// One block for a few tokens: scores, plan and placement in one launch.
template <int kPer, bool kSigmoid>
__global__ void __launch_bounds__(1024) moe_route_few_kernel(const MoeRouteParams p) {
  pdl_trigger();
  pdl_wait();
  __shared__ int warp_tot[32], counts[1024], at[1024];
  const int t = threadIdx.x;
  counts[t] = 0;
  for (int i = t; i < p.rows_cap; i += 1024) p.src_row[i] = -1;
  __syncthreads();
  for (int m = t >> 5; m < p.M; m += 32) moe_topk_row<kPer, kSigmoid>(p, m, t & 31, [&](int e) { atomicAdd(counts + e, 1); });
  __syncthreads();
  const int c = counts[t];
  int rows_total, tiles_total;
  const int off = block_excl_scan_1024((c + 15) & ~15, warp_tot, rows_total);
  const int toff = block_excl_scan_1024((c + p.nt - 1) / p.nt, warp_tot, tiles_total);
  at[t] = off;
  int i = toff;
  for (int r = 0; r < c; r += p.nt) p.tiles[i++] = make_int4(t, off + r, min(p.nt, c - r), 0);
  if (t == 0) {
    p.ntiles[0] = tiles_total;
    p.ntiles[1] = rows_total;
  }
  __syncthreads();
  for (int r = t; r < p.M * p.top_k; r += 1024) {
    const int le = p.topk_id[r] - p.e_lo;
    const bool mine = p.topk_id[r] >= 0 && le >= 0 && le < p.e_n;
    const int pos = mine ? atomicAdd(at + le, 1) : -1;
    p.slot_of[r] = pos;
    if (mine) p.src_row[pos] = r / p.top_k;
  }
}

// thread per route: claim a row in the expert's segment.
__global__ void moe_place_kernel(const MoeRouteParams p) {
  pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= p.M * p.top_k) return;
  const int le = p.topk_id[i] - p.e_lo;
  if (p.topk_id[i] < 0 || le < 0 || le >= p.e_n) { p.slot_of[i] = -1; return; }
  const int pos = p.offsets[le] + atomicAdd(p.cursors + le, 1);
  p.slot_of[i] = pos;
  p.src_row[pos] = i / p.top_k;
}

// block = K / 16 threads (one 16-byte chunk each); the CTAs stride over the LIVE rows (a device-side
// count): the grid is static (graph capture) but small, instead of one CTA per row of the worst case.
// to_fp8: the sorted rows feed MXFP4 experts, whose GEMM multiplies fp8 x fp8: an int8 value q (row scale s)
// leaves as e4m3(q * 448 / 127) with row scale s * 127 / 448 (round to nearest even, saturating).
__global__ void moe_gather_kernel(const int8_t* __restrict__ q, const float* __restrict__ scale, int M_pad,
                                  const int32_t* __restrict__ src_row, const int32_t* __restrict__ ntiles,
                                  int8_t* __restrict__ q_out, float* __restrict__ scale_out, int M_pad_out, int to_fp8) {
  pdl_trigger();
  pdl_wait();
  const int live = ntiles[1];
  const int kb = threadIdx.x >> 3, c = threadIdx.x & 7;       // k-block, logical 16-byte chunk
  for (int r = blockIdx.x; r < live; r += gridDim.x) {
    const int m = src_row[r];
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (m >= 0)
      v = *reinterpret_cast<const uint4*>(q + (static_cast<size_t>(kb) * M_pad + m) * 128 + ((c ^ (m & 7)) << 4));
    if (to_fp8) {
      uint32_t* w = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float f0 = static_cast<float>(static_cast<int8_t>(w[i] & 0xFFu)) * (448.f / 127.f);
        const float f1 = static_cast<float>(static_cast<int8_t>((w[i] >> 8) & 0xFFu)) * (448.f / 127.f);
        const float f2 = static_cast<float>(static_cast<int8_t>((w[i] >> 16) & 0xFFu)) * (448.f / 127.f);
        const float f3 = static_cast<float>(static_cast<int8_t>(w[i] >> 24)) * (448.f / 127.f);
        const uint32_t lo = __nv_cvt_float2_to_fp8x2(make_float2(f0, f1), __NV_SATFINITE, __NV_E4M3);
        const uint32_t hi = __nv_cvt_float2_to_fp8x2(make_float2(f2, f3), __NV_SATFINITE, __NV_E4M3);
        w[i] = lo | (hi << 16);
      }
    }
    *reinterpret_cast<uint4*>(q_out + (static_cast<size_t>(kb) * M_pad_out + r) * 128 + ((c ^ (r & 7)) << 4)) = v;
    if (threadIdx.x == 0) scale_out[r] = m >= 0 ? scale[m] * (to_fp8 ? 127.f / 448.f : 1.f) : 0.f;
  }
}

// grid = (ceil(H / 256), ceil(M / nt)), block 256: lane -> 8 columns, warp -> rows w, w + 8, ...
// out[m] = sum_k w[m,k] * y[slot_of[m,k]] (+ sigmoid(g[m]) * shared[m]), routes in top-k order.
__global__ void __launch_bounds__(256) moe_combine_kernel(const MoeCombineParams p) {
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = blockIdx.x * 256 + lane * 8;
  const int m0 = blockIdx.y * p.nt;
  const bool tp = p.tp_nranks > 1;
  uint32_t seq = 0, par = 0;
  if (tp) {
    seq = *p.tp_seq_base + static_cast<uint32_t>(p.tp_site) + 1u;
    par = seq & 1u;
  }
  if (n < p.H) {
    for (int r = warp; r < p.nt; r += 8) {
      const int m = m0 + r;
      if (m >= p.M) break;
      float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      for (int k = 0; k < p.top_k; ++k) {
        const int slot = p.slot_of[m * p.top_k + k];
        if (slot < 0) continue;
        const float w = p.topk_w[m * p.top_k + k];
        const uint4 raw = *reinterpret_cast<const uint4*>(p.y + static_cast<size_t>(slot) * p.H + n);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 f = __bfloat1622float2(h[i]);
          acc[2 * i] += w * f.x;
          acc[2 * i + 1] += w * f.y;
        }
      }
      if (p.shared) {
        float gs = 1.f;
        if (p.shared_gate) gs = 1.f / (1.f + __expf(-__bfloat162float(p.shared_gate[static_cast<size_t>(m) * p.ldg])));
        const uint4 raw = *reinterpret_cast<const uint4*>(p.shared + static_cast<size_t>(m) * p.H + n);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 f = __bfloat1622float2(h[i]);
          acc[2 * i] += gs * f.x;
          acc[2 * i + 1] += gs * f.y;
        }
      }
      uint4 o;
      __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
      for (int i = 0; i < 4; ++i) oh[i] = __floats2bfloat162_rn(acc[2 * i], acc[2 * i + 1]);
      if (tp) {
        const size_t off = ((static_cast<size_t>(par) * p.tp_nranks + p.tp_rank) * p.tp_rows + m) * p.tp_ld + n;
        for (int peer = 0; peer < p.tp_nranks; ++peer)
          *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.tp_recv[peer]) + off) = o;
      } else {
        *reinterpret_cast<uint4*>(p.out + static_cast<size_t>(m) * p.H + n) = o;
      }
    }
  }
  if (tp) {
    __threadfence_system();
    __syncthreads();
    if (threadIdx.x < p.tp_nranks) {
      const int tile_id = blockIdx.y * gridDim.x + blockIdx.x;
      uint32_t* f = p.tp_flags[threadIdx.x] + (static_cast<size_t>(par) * p.tp_nranks + p.tp_rank) * kMoeTpMaxTiles + tile_id;
      asm volatile("st.release.sys.global.u32 [%0], %1;" ::"l"(f), "r"(seq) : "memory");
    }
  }
}

}  // namespace saber

namespace saber {
static bool moe_few(const MoeRouteParams& p) { return p.logits_f32 != nullptr && p.M <= 64; }

template <int kPer, bool kSigmoid>
static int moe_route_form(const MoeRouteParams& p, cudaStream_t stream) {
  if (moe_few(p)) return static_cast<int>(launch(moe_route_few_kernel<kPer, kSigmoid>, dim3(1), dim3(1024), 0, stream, 2, p));
  launch(moe_topk_kernel<kPer, kSigmoid>, dim3((p.M + 7) / 8), dim3(256), 0, stream, 0, p);
  launch(moe_plan_kernel, dim3(1), dim3(1024), 0, stream, 0, p);
  launch(moe_place_kernel, dim3((p.M * p.top_k + 255) / 256), dim3(256), 0, stream, 0, p);
  return static_cast<int>(cudaGetLastError());
}
template <int kPer>
static int moe_route_go(const MoeRouteParams& p, cudaStream_t stream) {
  return p.sigmoid ? moe_route_form<kPer, true>(p, stream) : moe_route_form<kPer, false>(p, stream);
}
}  // namespace saber

extern "C" int saber_moe_route_launches(const saber::MoeRouteParams* p) { return saber::moe_few(*p) ? 1 : 3; }

extern "C" int saber_moe_route_launch(const saber::MoeRouteParams* p, cudaStream_t stream) {
  using namespace saber;
  if (p->sigmoid && p->logits_f32 == nullptr) return static_cast<int>(cudaErrorInvalidValue);
  if (p->E < 1 || p->E > 1024 || p->e_n > 1024 || p->top_k > kMoeMaxTopK || p->top_k < 1 || p->nt < 16 || (p->nt & 15) ||
      (p->groups > 1 && (p->E % p->groups || p->keep < 1 || p->keep * (p->E / p->groups) < p->top_k)))
    return static_cast<int>(cudaErrorInvalidValue);
  const int per = (p->E + 31) / 32;
  return per <= 1 ? moe_route_go<1>(*p, stream) : per <= 4 ? moe_route_go<4>(*p, stream) : per <= 16 ? moe_route_go<16>(*p, stream) : moe_route_go<32>(*p, stream);
}

extern "C" int saber_moe_gather_launch(const int8_t* q, const float* scale, int M_pad, const int32_t* src_row,
                                       const int32_t* ntiles, int8_t* q_out, float* scale_out, int rows_cap,
                                       int M_pad_out, int K, int to_fp8, cudaStream_t stream) {
  if ((K & 127) || K / 16 > 1024 || rows_cap > M_pad_out) return static_cast<int>(cudaErrorInvalidValue);
  saber::launch(saber::moe_gather_kernel, dim3(rows_cap < 1184 ? rows_cap : 1184), dim3(K / 16), 0, stream, 0, q, scale, M_pad, src_row, ntiles, q_out, scale_out, M_pad_out, to_fp8);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int saber_moe_combine_launch(const saber::MoeCombineParams* p, cudaStream_t stream) {
  if ((p->H & 7) || p->nt < 1) return static_cast<int>(cudaErrorInvalidValue);
  dim3 grid((p->H + 255) / 256, (p->M + p->nt - 1) / p->nt);
  if (p->tp_nranks > 1 &&
      (p->tp_nranks > 8 || static_cast<int>(grid.x * grid.y) > saber::kMoeTpMaxTiles || p->M > p->tp_rows || (p->tp_ld & 7)))
    return static_cast<int>(cudaErrorInvalidValue);
  saber::launch(saber::moe_combine_kernel, dim3(grid), dim3(256), 0, stream, 0, *p);
  return static_cast<int>(cudaGetLastError());
}
