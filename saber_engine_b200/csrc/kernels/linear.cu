// Linears around an fp32 residual stream.
//
// bf16: one tcgen05 GEMM kernel, token rows on the 128 accumulator lanes and 256 weight rows on the N
// side (the orientation and tile storage of gemm_i8.cu: pre-tiled operands, untiled bulk copies into a
// ring of stages, one MMA-issuing thread, eight epilogue warps).  Its epilogues keep the residual stream
// and the normalisation in fp32 without a kernel of their own: a "stream" linear adds its result to the
// fp32 row, writes the next linear's bf16 operand norm_w * x and the row's partial sums of squares; the
// next linear multiplies its result by the reciprocal root mean square.  A gated unit's activation is
// computed in the epilogue of its gate | up tiles.  Split-K parts go to a workspace and the last CTA of a
// tile to arrive adds them in order, so the result does not depend on the order of arrival.
//
// fp32: a CUDA-core GEMM (plain fused multiply-adds) followed by one row kernel that runs the same
// epilogue; the bf16 linear takes this two-launch form too when fuse = 0.
//
// A grouped product (mixtures of experts) is the same kernel over a table of row tiles, each against the weights of its
// expert.  Where the operand rows are tokens out of order, the eight epilogue warps, idle until the accumulator is done, copy them
// into the ring row by row (16-byte asynchronous copies, swizzled for their place in the tile).
#include "launch.cuh"
#include "linear.h"
#include "ptx_sm100.cuh"

namespace saber {

constexpr int kLinThreads = 320;
constexpr int kLinMaxStages = 8;
constexpr int kLinRow = 260;              // floats per staged accumulator row (16-byte accesses of eight lanes hit all banks)
constexpr uint32_t kLinTile = 32768;      // 256 weight rows x 64 bf16

__device__ __forceinline__ float clamped_glu(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit);
  const float u = fminf(fmaxf(up, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}

// A gated unit of act_kind 0, 4 or 5.
__device__ __forceinline__ float gated_unit(const LinEpi& e, float gate, float up) {
  if (e.act_kind == 4) return 0.5f * gate * (1.f + tanhf(0.79788456080286536f * fmaf(0.044715f * gate * gate, gate, gate))) * up;
  if (e.act_kind == 5) return gate / (1.f + expf(-gate)) * up;
  return clamped_glu(gate, up, e.limit, e.alpha);
}

__device__ __forceinline__ float relu_squared(float x) {
  const float r = fmaxf(x, 0.f);
  return r * r;
}

__device__ __forceinline__ float gelu(float x) { return 0.5f * x * (1.f + erff(x * 0.70710678118654752f)); }

__device__ __forceinline__ float stored(const LinEpi& e, int n, float v) {      // bias and cap of a stored column
  if (e.bias) v += e.bias[n];
  return e.cap > 0.f ? e.cap * tanhf(v / e.cap) : v;
}

constexpr int kGatedTile = 248;           // features of a tile of act_kind 2; row 248 of the tile is their gate

// x[i] (eight stream values of rows m + 8 i, columns from n on) += the sum over the rows' routes of weight times expert row.  A lane holds
// a route of each row; sixteen pieces of expert rows are requested together.
__device__ __forceinline__ void add_routes(const LinEpi& e, int m, int rows, int n, bool cols, int lane, float4 (&x)[4][2]) {
  int slot[4];
  float wt[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const bool in = 8 * i < rows && lane < e.routes;
    slot[i] = in ? e.slot_of[(m + 8 * i) * e.routes + lane] : -1;
    wt[i] = in ? e.route_w[(m + 8 * i) * e.routes + lane] : 0.f;
  }
  const __nv_bfloat16* y = static_cast<const __nv_bfloat16*>(e.y) + n;
  for (int k0 = 0; k0 < e.routes; k0 += 4) {
    uint4 q[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const int r = __shfl_sync(0xffffffffu, slot[i], (k0 + k) & 31);
        q[i][k] = make_uint4(0u, 0u, 0u, 0u);
        if (cols && r >= 0) q[i][k] = __ldcg(reinterpret_cast<const uint4*>(y + static_cast<size_t>(r) * e.ldy));
      }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float w = __shfl_sync(0xffffffffu, wt[i], (k0 + k) & 31);
        const uint4 u = q[i][k];
        float4& a = x[i][0];
        float4& b = x[i][1];
        a.x = fmaf(w, __uint_as_float(u.x << 16), a.x);
        a.y = fmaf(w, __uint_as_float(u.x & 0xFFFF0000u), a.y);
        a.z = fmaf(w, __uint_as_float(u.y << 16), a.z);
        a.w = fmaf(w, __uint_as_float(u.y & 0xFFFF0000u), a.w);
        b.x = fmaf(w, __uint_as_float(u.z << 16), b.x);
        b.y = fmaf(w, __uint_as_float(u.z & 0xFFFF0000u), b.y);
        b.z = fmaf(w, __uint_as_float(u.w << 16), b.z);
        b.w = fmaf(w, __uint_as_float(u.w & 0xFFFF0000u), b.w);
      }
  }
}

// reciprocal root mean square of the stream row behind operand row m (all lanes of a warp call together)
__device__ __forceinline__ float row_rms_scale(const LinEpi& e, int m, int lane) {
  if (e.ss == nullptr) return 1.f;
  float s = 0.f;
  for (int i = lane; i < e.ss_n; i += 32) s += __ldcg(e.ss + static_cast<size_t>(m) * e.ss_n + i);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  return 1.f / sqrtf(s * e.inv_width + e.eps);
}

// One finished row of a 256-column tile, by a warp.  acc(c): the eight (project, stream) or four (gated unit)
// accumulators from column c on.  sc: the row's scale (project); x0, x1: this lane's eight values of the stream row and what
// joins it (stream, when the linear adds to it), fetched by the caller ahead of time.
template <typename Acc>
__device__ __forceinline__ void linear_row_epilogue(const LinEpi& e, const Acc& acc, int m, int tile_n, int lane, float sc, float4 x0, float4 x1) {
  const int n0 = tile_n * 256;
  if (!e.stream) {
    if (tile_n < e.lat_tiles) {
      const int n = n0 + lane * 8;
      const float4 a = acc(lane * 8), b = acc(lane * 8 + 4);
      const float v[8] = {a.x * sc, a.y * sc, a.z * sc, a.w * sc, b.x * sc, b.y * sc, b.z * sc, b.w * sc};
      float y[8], sq = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const bool in = n + j < e.lat_n;
        sq += in ? v[j] * v[j] : 0.f;
        y[j] = in ? v[j] * e.lat_w[n + j] : 0.f;
      }
      if (n < e.lat.ld) operand_store8(e.lat, m, n, y);              // (the operand ends at a multiple of 64 columns)
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
      const int g = tile_n * 2 + (lane >> 4);
      if ((lane & 15) == 0 && g < e.lat_ss_n) e.lat_ss[static_cast<size_t>(m) * e.lat_ss_n + g] = sq;
      return;
    }
    if (tile_n < e.act_tile0) {
      const int n = n0 + lane * 8;
      if (n >= e.n_plain) return;
      float4 a = acc(lane * 8), b = acc(lane * 8 + 4);
      if (e.out_bf16) {                                              // (rows of whole groups of eight)
        const float v[8] = {a.x * sc, a.y * sc, a.z * sc, a.w * sc, b.x * sc, b.y * sc, b.z * sc, b.w * sc};
        uint4 q;
        uint32_t* u = reinterpret_cast<uint32_t*>(&q);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
          u[j] = *reinterpret_cast<const uint32_t*>(&h);
        }
        *reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(e.out) + static_cast<size_t>(m) * e.ldo + n) = q;
        return;
      }
      float* o = e.out + static_cast<size_t>(m) * e.ldo + n;
      a = make_float4(a.x * sc, a.y * sc, a.z * sc, a.w * sc);
      b = make_float4(b.x * sc, b.y * sc, b.z * sc, b.w * sc);
      if (n + 8 <= e.n_plain && !(e.cap > 0.f)) {
        if (e.bias) {
          const float4 c = *reinterpret_cast<const float4*>(e.bias + n), d = *reinterpret_cast<const float4*>(e.bias + n + 4);
          a = make_float4(a.x + c.x, a.y + c.y, a.z + c.z, a.w + c.w);
          b = make_float4(b.x + d.x, b.y + d.y, b.z + d.z, b.w + d.w);
        }
        *reinterpret_cast<float4*>(o) = a;
        *reinterpret_cast<float4*>(o + 4) = b;
      } else {
        const float v[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
        for (int j = 0; j < 8; ++j)
          if (n + j < e.n_plain) o[j] = stored(e, n + j, v[j]);
      }
    } else if (e.act_kind == 1) {
      const float4 a = acc(lane * 8), b = acc(lane * 8 + 4);
      const float y[8] = {relu_squared(a.x * sc), relu_squared(a.y * sc), relu_squared(a.z * sc), relu_squared(a.w * sc),
                          relu_squared(b.x * sc), relu_squared(b.y * sc), relu_squared(b.z * sc), relu_squared(b.w * sc)};
      const int k = e.act_k0 + (tile_n - e.act_tile0) * 256 + lane * 8;
      if (k < e.act.ld) operand_store8(e.act, m, k, y);              // (the operand ends at a multiple of 64 columns, the tile of 256)
    } else if (e.act_kind == 2) {
      const float4 a = acc(lane * 8), b = acc(lane * 8 + 4);
      const float gate = 1.f / (1.f + expf(-__shfl_sync(0xffffffffu, a.x * sc, 31)));
      const float y[8] = {gate * relu_squared(a.x * sc), gate * relu_squared(a.y * sc), gate * relu_squared(a.z * sc), gate * relu_squared(a.w * sc),
                          gate * relu_squared(b.x * sc), gate * relu_squared(b.y * sc), gate * relu_squared(b.z * sc), gate * relu_squared(b.w * sc)};
      const int k = e.act_k0 + (tile_n - e.act_tile0) * kGatedTile + lane * 8;
      if (lane < 31 && k < e.act.ld) operand_store8(e.act, m, k, y);
    } else if (e.act_kind == 3) {
      const float4 a = acc(lane * 8), b = acc(lane * 8 + 4);
      const int f = (tile_n - e.act_tile0) * 256 + lane * 8, k = e.act_k0 + f;
      if (k >= e.act.ld) return;
      float4 c = make_float4(0.f, 0.f, 0.f, 0.f), d = c;
      if (e.act_bias) {
        c = *reinterpret_cast<const float4*>(e.act_bias + f);
        d = *reinterpret_cast<const float4*>(e.act_bias + f + 4);
      }
      const float y[8] = {gelu(fmaf(a.x, sc, c.x)), gelu(fmaf(a.y, sc, c.y)), gelu(fmaf(a.z, sc, c.z)), gelu(fmaf(a.w, sc, c.w)),
                          gelu(fmaf(b.x, sc, d.x)), gelu(fmaf(b.y, sc, d.y)), gelu(fmaf(b.z, sc, d.z)), gelu(fmaf(b.w, sc, d.w))};
      operand_store8(e.act, m, k, y);
    } else {
      const float4 g = acc(lane * 4), u = acc(128 + lane * 4);
      operand_store4(e.act, m, e.act_k0 + (tile_n - e.act_tile0) * 128 + lane * 4,
                     make_float4(gated_unit(e, g.x * sc, u.x * sc), gated_unit(e, g.y * sc, u.y * sc), gated_unit(e, g.z * sc, u.z * sc),
                                 gated_unit(e, g.w * sc, u.w * sc)));
    }
    return;
  }
  const int n = n0 + lane * 8;
  float sq = 0.f;
  if (n < e.width) {                              // ldx is a multiple of 32: whole groups of eight are in bounds
    float* xr = e.x + static_cast<size_t>(m) * e.ldx + n;
    const float4 a = acc(lane * 8), b = acc(lane * 8 + 4);
    float v[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
    if (e.add) {
      v[0] += x0.x; v[1] += x0.y; v[2] += x0.z; v[3] += x0.w;
      v[4] += x1.x; v[5] += x1.y; v[6] += x1.z; v[7] += x1.w;
    }
    float y[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const bool in = n + j < e.width;
      if (e.bias && in) v[j] += e.bias[n + j];
      sq += v[j] * v[j];
      y[j] = e.norm_w ? (in ? v[j] * e.norm_w[n + j] : 0.f) : v[j];
    }
    *reinterpret_cast<float4*>(xr) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(xr + 4) = make_float4(v[4], v[5], v[6], v[7]);
    operand_store8(e.op, m, e.op_k0 + n, y);
    if (e.norm_w2 != nullptr) {
#pragma unroll
      for (int j = 0; j < 8; ++j) y[j] = n + j < e.width ? v[j] * e.norm_w2[n + j] : 0.f;
      operand_store8(e.op2, m, n, y);
    }
  }
  if (e.ss_out == nullptr) return;
#pragma unroll
  for (int o = 8; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);       // per half warp: 128 columns
  const int g = tile_n * 2 + (lane >> 4);
  if ((lane & 15) == 0 && g < e.ss_out_n) e.ss_out[static_cast<size_t>(m) * e.ss_out_n + g] = sq;
}

// The staged rows of a tile (shared memory, kLinRow floats apart), four per warp and round: their stream rows are
// requested together.
__device__ __forceinline__ void linear_tile_epilogue(const LinEpi& e, const float* tile_s, const float* scale_s, int mb, int rows, int tile_n,
                                                     int w, int lane) {
  const int n = tile_n * 256 + lane * 8;
  const bool addx = e.stream && e.add && n < e.width;
  for (int r0 = w; r0 < rows; r0 += 32) {
    float4 x[4][2];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = r0 + 8 * i;
      x[i][0] = x[i][1] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (addx && r < rows) {
        const float4* xr = reinterpret_cast<const float4*>(e.x + static_cast<size_t>(mb + r) * e.ldx + n);
        x[i][0] = __ldcg(xr);                     // (what joins it may come from the CTA of another part)
        x[i][1] = __ldcg(xr + 1);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = r0 + 8 * i;
      if (r < rows)
        linear_row_epilogue(e, [&](int c) { return *reinterpret_cast<const float4*>(tile_s + r * kLinRow + c); }, mb + r, tile_n, lane,
                            scale_s[r], x[i][0], x[i][1]);
    }
  }
}

// The routed rows of a tile join its stream rows in memory while the main loop runs (the epilogue then reads them there).
__device__ __forceinline__ void linear_tile_routes(const LinEpi& e, int mb, int rows, int tile_n, int w, int lane) {
  const int n = tile_n * 256 + lane * 8;
  for (int r0 = w; r0 < rows; r0 += 32) {
    float4 x[4][2];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      x[i][0] = x[i][1] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (n < e.width && r0 + 8 * i < rows) {
        const float4* xr = reinterpret_cast<const float4*>(e.x + static_cast<size_t>(mb + r0 + 8 * i) * e.ldx + n);
        x[i][0] = __ldcg(xr);
        x[i][1] = __ldcg(xr + 1);
      }
    }
    add_routes(e, mb + r0, rows - r0, n, n < e.width, lane, x);
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (n < e.width && r0 + 8 * i < rows) {
        float4* xr = reinterpret_cast<float4*>(e.x + static_cast<size_t>(mb + r0 + 8 * i) * e.ldx + n);
        __stcg(xr, x[i][0]);
        __stcg(xr + 1, x[i][1]);
      }
  }
}

// kGroup: 0 a plain product, 1 a grouped one, 2 a grouped one whose operand rows are gathered by the epilogue warps
template <int kMT, int kGroup>
__global__ void __launch_bounds__(kLinThreads, 1) lin_bf16_kernel(const __grid_constant__ LinParams p, const int stages) {
  extern __shared__ uint8_t smem_raw[];
  // one round of CTAs: the successor may take the SMs this grid leaves idle or frees (until its own wait it touches
  // weights only)
  if (kGroup != 0 || gridDim.x == 1) pdl_trigger();
  int4 group = make_int4(0, 0, 0, 0);
  if constexpr (kGroup != 0) {
    pdl_wait();
    if (static_cast<int>(blockIdx.x) >= p.group_ntiles[0]) return;
    group = p.group_tiles[blockIdx.x];
  }
  __shared__ uint64_t bars[2 * kLinMaxStages + 1];
  __shared__ uint32_t tmem_base_s, is_last_s, abort_s;
  __shared__ float scale_s[256];

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile_m = blockIdx.x, tile_n = blockIdx.y, split = blockIdx.z;
  const int KB = p.K >> 6;
  const int kb_per = (KB + p.splits - 1) / p.splits;
  const int kb0 = split * kb_per;
  const int nkb = min(KB, kb0 + kb_per) - kb0;        // host guarantees >= 1
  const int m0 = kGroup != 0 ? group.y : tile_m * p.nt * kMT;
  const int m_end = kGroup != 0 ? group.y + group.z : p.M;
  const uint32_t abytes = static_cast<uint32_t>(p.nt) * 128u * kMT;
  const uint32_t a_smem = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t w_smem = a_smem + static_cast<uint32_t>(stages) * abytes;
  const uint32_t bar_full = smem_u32(&bars[0]);
  const uint32_t bar_empty = smem_u32(&bars[kLinMaxStages]);
  const uint32_t bar_acc = smem_u32(&bars[2 * kLinMaxStages]);
  constexpr uint32_t kCols = kMT == 2 ? 512u : 256u;

  if (threadIdx.x == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(bar_full + 8 * s, kGroup == 2 ? 9 : 1);
      mbar_init(bar_empty + 8 * s, 1);
    }
    mbar_init(bar_acc, 1);
    abort_s = 0;
    is_last_s = 1;
    mbar_init_fence();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_base_s), kCols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_d = tmem_base_s;

  if (warp == 0) {
    // ---------------------------------------------------------------- producer
    if (lane == 0) {
      constexpr bool kCopyA = kGroup != 2;
      const uint32_t acopy = kGroup == 0 ? abytes : static_cast<uint32_t>((group.z + 7) & ~7) * 128u;   // a group's own rows
      const uint32_t tx = kLinTile + (kCopyA ? acopy : 0u);
      const uint64_t pol = gridDim.x > 1 ? l2_policy_evict_normal() : l2_policy_evict_first();
      const uint8_t* wp = static_cast<const uint8_t*>(p.w) + group.x * p.group_w_stride + (static_cast<size_t>(tile_n) * KB + kb0) * kLinTile;
      const uint8_t* ap = static_cast<const uint8_t*>(p.a2 != nullptr && tile_n >= p.a2_tile0 ? p.a2 : p.a) +
                          (static_cast<size_t>(kb0) * p.M_pad + m0) * 128;
      const size_t a_step = static_cast<size_t>(p.M_pad) * 128;
      const int pre = min(stages, nkb);
      for (int it = 0; it < pre; ++it) {         // weights do not depend on the predecessor kernel
        mbar_arrive_expect_tx(bar_full + 8 * it, tx);
        bulk_g2s_hint(w_smem + it * kLinTile, wp, kLinTile, bar_full + 8 * it, pol);
        wp += kLinTile;
      }
      pdl_wait();
      if constexpr (kCopyA)
        for (int it = 0; it < pre; ++it) {
          bulk_g2s(a_smem + it * abytes, ap, acopy, bar_full + 8 * it);
          ap += a_step;
        }
      int issued = pre, s = pre == stages ? 0 : pre;
      uint32_t ph = pre == stages ? 1u : 0u;
      bool ok = true;
      for (int it = pre; it < nkb; ++it) {
        if (!mbar_wait(bar_empty + 8 * s, ph ^ 1u, p.err, kErrWaitEmpty)) { ok = false; break; }
        mbar_arrive_expect_tx(bar_full + 8 * s, tx);
        bulk_g2s_hint(w_smem + s * kLinTile, wp, kLinTile, bar_full + 8 * s, pol);
        if constexpr (kCopyA) bulk_g2s(a_smem + s * abytes, ap, acopy, bar_full + 8 * s);
        wp += kLinTile;
        ap += a_step;
        issued = it + 1;
        if (++s == stages) { s = 0; ph ^= 1u; }
      }
      if (!ok)                                   // do not leave while an own copy is in flight
        for (int it = max(0, issued - stages); it < issued; ++it)
          mbar_wait(bar_full + 8 * (it % stages), (it / stages) & 1, p.err, kErrWaitDrain);
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      const uint32_t idesc = make_idesc(kCFmtF32, kFmtBF16, kFmtBF16, 128, 256);
      const uint64_t desc_hi = make_desc_k128(0);
      uint32_t a_addr = a_smem;
      int s = 0;
      uint32_t ph = 0;
      bool ok = true;
      for (int it = 0; it < nkb; ++it) {
        if (!mbar_wait(bar_full + 8 * s, ph, p.err, kErrWaitReady)) { ok = false; break; }
        tc_fence_after_sync();
        const uint32_t w_addr = w_smem + s * kLinTile;
        const uint64_t a_desc = desc_hi | static_cast<uint64_t>((a_addr & 0x3FFFFu) >> 4);
        const uint64_t b_desc = desc_hi | static_cast<uint64_t>((w_addr & 0x3FFFFu) >> 4);
#pragma unroll
        for (int j2 = 0; j2 < kMT; ++j2) {
          if (kGroup != 0 && j2 > 0 && j2 * p.nt >= group.z) break;
          const uint32_t dj = tmem_d + static_cast<uint32_t>(j2) * 256u;
          const uint64_t aj = a_desc + static_cast<uint64_t>(j2) * (static_cast<uint64_t>(p.nt) * 128u >> 4);
          mma_f16_ss(dj, aj, b_desc, idesc, it != 0 ? 1u : 0u);
          mma_f16_ss(dj, aj + 2, b_desc + 2, idesc, 1u);
          mma_f16_ss(dj, aj + 4, b_desc + 4, idesc, 1u);
          mma_f16_ss(dj, aj + 6, b_desc + 6, idesc, 1u);
        }
        mma_commit(bar_empty + 8 * s);
        a_addr += abytes;
        if (++s == stages) { s = 0; ph ^= 1u; a_addr = a_smem; }
      }
      mma_commit(bar_acc);
      if (!ok) mbar_wait(bar_acc, 0, nullptr, 0);   // issued MMAs retire before the tensor memory is freed
    }
  } else {
    // ---------------------------------------------------------------- epilogue (8 warps)
    // The accumulator arrives a row per lane; it is staged in shared memory (the operand ring is idle by then) so
    // that a warp finishes a whole 256-column row at a time with contiguous global accesses.
    const int te = threadIdx.x - 64;              // 0..255
    const int grp = te >> 7;                      // column half this warp reads out
    const int q4 = warp & 3;                      // TMEM lane quarter of this warp
    const LinEpi& e = p.e;
    pdl_wait();
    if constexpr (kGroup == 2) {
      // operand rows: up to 4 kMT 16-byte pieces of every k-block per thread
      constexpr int kLag = kMT == 2 ? 1 : 2;      // (two below the number of stages: the tensor cores always have a k-block)
      constexpr int kPieces = 4 * kMT;
      const uint8_t* src[kPieces];
      uint32_t dst[kPieces];
      bool live[kPieces];
      const size_t a_step = static_cast<size_t>(p.M_pad) * 128;
#pragma unroll
      for (int i = 0; i < kPieces; ++i) {
        const int r = (te + 256 * i) >> 3, c = te & 7;
        live[i] = r < group.z;
        const int m = live[i] ? max(p.src_row[m0 + r], 0) : 0;
        src[i] = static_cast<const uint8_t*>(p.a) + static_cast<size_t>(m) * 128 + (((c ^ m) & 7) << 4);
        dst[i] = a_smem + static_cast<uint32_t>(r) * 128u + (((c ^ r) & 7) << 4);
      }
      int s = 0, done = 0;                        // done: k-blocks handed to the tensor cores
      uint32_t ph = 0;
      bool ok = true;
      auto hand_over = [&](int it) {
        fence_proxy_async_smem();
        __syncwarp();
        if (lane == 0) mbar_arrive(bar_full + 8 * (it % stages));
      };
      for (int it = 0; it < nkb; ++it) {
        if (it >= stages) ok = __all_sync(0xffffffffu, mbar_wait(bar_empty + 8 * s, ph ^ 1u, p.err, kErrWaitEmpty));
        if (!ok) break;
#pragma unroll
        for (int i = 0; i < kPieces; ++i) {
          if (live[i]) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst[i] + s * abytes), "l"(src[i]) : "memory");
          src[i] += a_step;
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (it >= kLag) {
          asm volatile("cp.async.wait_group %0;" ::"n"(kLag) : "memory");
          hand_over(done++);
        }
        if (++s == stages) { s = 0; ph ^= 1u; }
      }
      asm volatile("cp.async.wait_group 0;" ::: "memory");
      if (ok)
        while (done < nkb) hand_over(done++);
    }
    // row scales while the main loop runs: a thread per row
    if (te < p.nt * kMT) {
      float sc = 1.f;
      if (e.ss != nullptr && m0 + te < m_end) {
        const float* q = e.ss + static_cast<size_t>(kGroup == 2 ? max(p.src_row[m0 + te], 0) : m0 + te) * e.ss_n;
        float s = 0.f;
#pragma unroll 8
        for (int i = 0; i < e.ss_n; ++i) s += __ldcg(q + i);
        sc = 1.f / sqrtf(s * e.inv_width + e.eps);
      }
      scale_s[te] = sc;
    }
    if constexpr (kGroup == 0)
      if (e.y != nullptr && split == 0)
        for (int j2 = 0; j2 < kMT; ++j2) linear_tile_routes(e, m0 + j2 * p.nt, min(p.nt, p.M - m0 - j2 * p.nt), tile_n, warp - 2, lane);
    bool ok = mbar_wait(bar_acc, 0, p.err, kErrWaitAcc);
    if (!ok) abort_s = 1u;
    named_bar_sync(1, 256);
    ok = abort_s == 0u;
    tc_fence_after_sync();
    const int rowl = q4 * 32 + lane;
    const uint32_t t_lane = tmem_d + (static_cast<uint32_t>(q4 * 32) << 16);
    const int tile_lin = tile_m * gridDim.y + tile_n;
    float* tile_s = reinterpret_cast<float*>(smem_raw + (a_smem - smem_u32(smem_raw)));
    if (p.splits > 1) {                           // (kMT == 1)
      const int mt = min(p.nt, m_end - m0);
      float* part = p.ws + (static_cast<size_t>(tile_lin) * p.splits + split) * p.nt * 256;
      if (ok && q4 * 32 < mt) {
        for (int c = grp * 128; c < grp * 128 + 128; c += 32) {
          uint32_t r[32];
          tmem_ld32(t_lane + c, r);
          tmem_ld_wait();
          if (rowl < mt) {
#pragma unroll
            for (int j = 0; j < 8; ++j)
              __stcg(reinterpret_cast<float4*>(part + (static_cast<size_t>((c >> 2) + j) * p.nt + rowl) * 4),
                     make_float4(__uint_as_float(r[4 * j]), __uint_as_float(r[4 * j + 1]), __uint_as_float(r[4 * j + 2]),
                                 __uint_as_float(r[4 * j + 3])));
          }
        }
      }
      __threadfence();
      named_bar_sync(1, 256);
      if (te == 0) {
        const uint32_t old = atomicAdd(p.counters + tile_lin, 1u);
        const bool last = old == static_cast<uint32_t>(p.splits) - 1u;
        if (last) p.counters[tile_lin] = 0u;
        __threadfence();
        is_last_s = last ? 1u : 0u;
      }
      named_bar_sync(1, 256);
      if (!is_last_s) ok = false;
      __threadfence();
      if (ok) {                                   // the parts in order, a 16-byte group per thread
        const float* parts = p.ws + static_cast<size_t>(tile_lin) * p.splits * p.nt * 256;
        const size_t step = static_cast<size_t>(p.nt) * 256;
        for (int i = te; i < 64 * mt; i += 256) {
          const int c4 = i / mt, r = i - c4 * mt;
          const float* src = parts + (static_cast<size_t>(c4) * p.nt + r) * 4;
          float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
          for (int sp = 0; sp < p.splits; ++sp) {
            const float4 f = __ldcg(reinterpret_cast<const float4*>(src + sp * step));
            s.x += f.x; s.y += f.y; s.z += f.z; s.w += f.w;
          }
          *reinterpret_cast<float4*>(tile_s + r * kLinRow + c4 * 4) = s;
        }
        named_bar_sync(1, 256);
        linear_tile_epilogue(e, tile_s, scale_s, m0, mt, tile_n, warp - 2, lane);
      }
    } else if (ok) {
#pragma unroll 1
      for (int j2 = 0; j2 < kMT; ++j2) {
        const int mb = m0 + j2 * p.nt;
        const int mt = min(p.nt, m_end - mb);
        if (mt <= 0) break;                       // uniform
        if (j2 > 0) named_bar_sync(1, 256);
        if (q4 * 32 < mt) {
          for (int c = grp * 128; c < grp * 128 + 128; c += 32) {
            uint32_t r[32];
            tmem_ld32(t_lane + static_cast<uint32_t>(j2) * 256u + c, r);
            tmem_ld_wait();
            if (rowl < mt) {
#pragma unroll
              for (int j = 0; j < 8; ++j)
                *reinterpret_cast<float4*>(tile_s + rowl * kLinRow + c + 4 * j) =
                    make_float4(__uint_as_float(r[4 * j]), __uint_as_float(r[4 * j + 1]), __uint_as_float(r[4 * j + 2]), __uint_as_float(r[4 * j + 3]));
            }
          }
        }
        named_bar_sync(1, 256);
        linear_tile_epilogue(e, tile_s, scale_s + j2 * p.nt, mb, mt, tile_n, warp - 2, lane);
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_d, kCols);
}

// ------------------------------------------------------------------------------------ fp32 GEMM
// 64 x 64 output tile, 16 k per step, 4 x 4 outputs per thread; plain fused multiply-adds.
__global__ void __launch_bounds__(256) lin_f32_kernel(const __grid_constant__ LinParams p) {
  pdl_wait();
  __shared__ float as[16][68], ws[16][68];
  const int N = p.N_pad, K = p.K, n0 = blockIdx.x * 64;
  int m0 = blockIdx.y * 64, m_end = p.M;
  const float* w = static_cast<const float*>(p.w);
  const float* a = static_cast<const float*>(p.a2 != nullptr && n0 >= p.a2_tile0 * 256 ? p.a2 : p.a);
  if (p.group_tiles != nullptr) {
    if (static_cast<int>(blockIdx.y) >= p.group_ntiles[0]) return;
    const int4 g = p.group_tiles[blockIdx.y];
    m0 = g.y;
    m_end = g.y + g.z;
    w += g.x * (p.group_w_stride / sizeof(float));
  }
  float* out = p.ws;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
  float acc[4][4] = {};
  const bool live = m0 + lr < m_end;
  const int row = live && p.src_row != nullptr ? max(p.src_row[m0 + lr], 0) : m0 + lr;
  for (int k0 = 0; k0 < K; k0 += 16) {
    const float4 av = live ? *reinterpret_cast<const float4*>(a + static_cast<size_t>(row) * K + k0 + lk) : make_float4(0, 0, 0, 0);
    const float4 wv = *reinterpret_cast<const float4*>(w + static_cast<size_t>(n0 + lr) * K + k0 + lk);   // N is a multiple of 256
    as[lk][lr] = av.x; as[lk + 1][lr] = av.y; as[lk + 2][lr] = av.z; as[lk + 3][lr] = av.w;
    ws[lk][lr] = wv.x; ws[lk + 1][lr] = wv.y; ws[lk + 2][lr] = wv.z; ws[lk + 3][lr] = wv.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { x[i] = as[k][ty * 4 + i]; y[i] = ws[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m < m_end)
      *reinterpret_cast<float4*>(out + static_cast<size_t>(m) * N + n0 + tx * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
  }
}

// The same epilogue from the product rows [M][N_pad]: one CTA of eight warps per row.
__global__ void __launch_bounds__(256) lin_epi_kernel(const __grid_constant__ LinParams p) {
  pdl_wait();
  const LinEpi& e = p.e;
  const int m = blockIdx.x;
  const float* acc = p.ws + static_cast<size_t>(m) * p.N_pad;
  int token = m;
  if (p.group_tiles != nullptr) {                   // padding between the experts' rows: rows of no token
    token = p.group_rows[m];
    if (token < 0) return;
  }
  if (!e.stream) {
    const float sc = row_rms_scale(e, p.src_row != nullptr ? token : m, threadIdx.x & 31);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int g = warp; g < e.lat_tiles * 2; g += 8) {
      float sq = 0.f;
      for (int n = g * 128 + lane; n < min(e.lat_n, g * 128 + 128); n += 32) {
        const float v = acc[n] * sc;
        sq += v * v;
        operand_store1(e.lat, m, n, v * e.lat_w[n]);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
      if (lane == 0 && g < e.lat_ss_n) e.lat_ss[static_cast<size_t>(m) * e.lat_ss_n + g] = sq;
    }
    for (int n = e.lat_tiles * 256 + threadIdx.x; n < e.n_plain; n += 256) {
      const size_t at = static_cast<size_t>(m) * e.ldo + n;
      if (e.out_bf16) reinterpret_cast<__nv_bfloat16*>(e.out)[at] = __float2bfloat16(acc[n] * sc);
      else e.out[at] = stored(e, n, acc[n] * sc);
    }
    const int tiles = p.N_pad / 256;
    if (e.act_kind == 2) {
      for (int i = threadIdx.x; i < min((tiles - e.act_tile0) * kGatedTile, e.act.ld - e.act_k0); i += 256) {
        const float* t = acc + static_cast<size_t>(e.act_tile0 + i / kGatedTile) * 256;
        operand_store1(e.act, m, e.act_k0 + i, relu_squared(t[i % kGatedTile] * sc) / (1.f + expf(-t[kGatedTile] * sc)));
      }
      return;
    }
    if (e.act_kind == 3) {
      for (int i = threadIdx.x; i < min((tiles - e.act_tile0) * 256, e.act.ld - e.act_k0); i += 256)
        operand_store1(e.act, m, e.act_k0 + i, gelu(fmaf(acc[e.act_tile0 * 256 + i], sc, e.act_bias ? e.act_bias[i] : 0.f)));
      return;
    }
    if (e.act_kind == 1) {
      for (int i = threadIdx.x; i < min((tiles - e.act_tile0) * 256, e.act.ld - e.act_k0); i += 256)
        operand_store1(e.act, m, e.act_k0 + i, relu_squared(acc[e.act_tile0 * 256 + i] * sc));
      return;
    }
    for (int i = threadIdx.x; i < (tiles - e.act_tile0) * 128; i += 256) {
      const float* t = acc + static_cast<size_t>(e.act_tile0 + (i >> 7)) * 256 + (i & 127);
      operand_store1(e.act, m, e.act_k0 + i, gated_unit(e, t[0] * sc, t[128] * sc));
    }
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, groups = (e.width + 127) / 128;
  for (int g = warp; g < groups; g += 8) {
    float sq = 0.f;
    for (int n = g * 128 + lane; n < min(e.width, g * 128 + 128); n += 32) {
      float* xr = e.x + static_cast<size_t>(m) * e.ldx + n;
      float y = acc[n] + (e.bias ? e.bias[n] : 0.f);
      if (e.y != nullptr)
        for (int k = 0; k < e.routes; ++k) {
          const int r = e.slot_of[m * e.routes + k];
          if (r < 0) continue;
          const size_t at = static_cast<size_t>(r) * e.ldy + n;
          y = fmaf(e.route_w[m * e.routes + k], e.y_f32 ? static_cast<const float*>(e.y)[at] : __bfloat162float(static_cast<const __nv_bfloat16*>(e.y)[at]), y);
        }
      const float v = (e.add ? *xr : 0.f) + y;
      *xr = v;
      sq += v * v;
      operand_store1(e.op, m, e.op_k0 + n, e.norm_w ? v * e.norm_w[n] : v);
      if (e.norm_w2 != nullptr) operand_store1(e.op2, m, n, v * e.norm_w2[n]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    if (lane == 0 && e.ss_out != nullptr) e.ss_out[static_cast<size_t>(m) * e.ss_out_n + g] = sq;
  }
}

// ------------------------------------------------------------------------------------ stream rows
__global__ void __launch_bounds__(256) stream_embed_kernel(const __grid_constant__ StreamEmbedParams p) {
  pdl_wait();
  const int m = blockIdx.x;
  const int id = min(max(p.ids[m], 0), p.vocab - 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int g = warp; g * 128 < p.width; g += 8) {
    float sq = 0.f;
    for (int n = g * 128 + lane; n < min(p.width, g * 128 + 128); n += 32) {
      const size_t i = static_cast<size_t>(id) * p.width + n;
      const float t = p.table_f32 ? static_cast<const float*>(p.table)[i] : __bfloat162float(static_cast<const __nv_bfloat16*>(p.table)[i]);
      const float v = t * p.scale;
      p.x[static_cast<size_t>(m) * ((p.width + 31) / 32 * 32) + n] = v;
      sq += v * v;
      if (p.x0_k0 >= 0) operand_store1(p.x0, m, p.x0_k0 + n, v);
      operand_store1(p.op, m, p.op_k0 + n, p.norm_w ? v * p.norm_w[n] : v);
      if (p.norm_w2 != nullptr) operand_store1(p.op2, m, n, v * p.norm_w2[n]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    if (lane == 0 && p.ss_out != nullptr) p.ss_out[static_cast<size_t>(m) * p.ss_out_n + g] = sq;
  }
}

__global__ void __launch_bounds__(256) stream_norm_kernel(const __grid_constant__ StreamNormParams p) {
  pdl_wait();
  __shared__ float red[8];
  const int i = blockIdx.x;
  const float* x = p.x + static_cast<size_t>(p.rows ? p.rows[i] : i) * p.ldx;
  float sq = 0.f;
  for (int n = threadIdx.x; n < p.width; n += 256) sq += x[n] * x[n];
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
  __syncthreads();
  sq = 0.f;
  for (int w = 0; w < 8; ++w) sq += red[w];
  const float r = 1.f / sqrtf(sq / static_cast<float>(p.width) + p.eps);
  for (int n = threadIdx.x; n < p.width; n += 256) operand_store1(p.op, i, n, x[n] * r * p.w[n]);
}

}  // namespace saber

extern "C" int saber_linear_launches(const saber::LinParams* p) { return (p->fp32 || !p->fuse) ? 2 : 1; }

extern "C" int saber_linear_launch(const saber::LinParams* p, cudaStream_t stream) {
  using namespace saber;
  const LinEpi& e = p->e;
  if (p->M <= 0 || (p->N_pad & 255) || (p->K & 63) || p->K <= 0 || (p->M > p->M_pad && p->group_tiles == nullptr)) return static_cast<int>(cudaErrorInvalidValue);
  if (e.y != nullptr && (!e.stream || !e.add || e.routes < 1 || e.routes > 32 || e.slot_of == nullptr || e.route_w == nullptr || e.y_f32 != p->fp32 || (e.ldy & 7)))
    return static_cast<int>(cudaErrorInvalidValue);
  if (e.stream ? (e.width > p->N_pad || (e.ldx & 31) || e.x == nullptr)
               : (e.n_plain > e.act_tile0 * 256 || e.act_tile0 * 256 > p->N_pad || (e.ldo & 3)))
    return static_cast<int>(cudaErrorInvalidValue);
  const bool grouped = p->group_tiles != nullptr;
  if (grouped && (p->group_ntiles == nullptr || p->group_rows == nullptr || p->group_max < 1 || p->splits != 1 || e.stream || p->a2 != nullptr ||
                  (p->src_row != nullptr && p->src_row != p->group_rows)))
    return static_cast<int>(cudaErrorInvalidValue);
  if (!e.stream && (e.lat_tiles > e.act_tile0 || e.lat_n > e.lat_tiles * 256 || (e.out_bf16 && (e.n_plain & 7)))) return static_cast<int>(cudaErrorInvalidValue);
  if (p->fp32) {
    cudaError_t r = launch(lin_f32_kernel, dim3(p->N_pad / 64, grouped ? p->group_max : (p->M + 63) / 64), dim3(256), 0, stream, 0, *p);
    if (r != cudaSuccess) return static_cast<int>(r);
    return static_cast<int>(launch(lin_epi_kernel, dim3(p->M), dim3(256), 0, stream, 0, *p));
  }
  if (p->nt < 16 || p->nt > 128 || (p->nt & 15) || (p->M_pad % p->nt && !grouped) || p->splits < 1) return static_cast<int>(cudaErrorInvalidValue);
  const int KB = p->K >> 6;
  const int kb_per = (KB + p->splits - 1) / p->splits;
  if ((p->splits - 1) * kb_per >= KB) return static_cast<int>(cudaErrorInvalidValue);
  LinParams q = *p;
  if (!p->fuse) {
    // product rows only: the split parts use the workspace behind them
    q.e = LinEpi{};
    q.e.out = p->ws;
    q.e.ldo = p->N_pad;
    q.e.n_plain = p->N_pad;
    q.e.act_tile0 = p->N_pad / 256;
    q.ws = p->ws + static_cast<size_t>(p->M) * p->N_pad;
  }
  static bool ready[64];
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return static_cast<int>(cudaErrorInvalidDevice);
  constexpr int kSmem = 224 * 1024;
  if (!ready[dev]) {
    cudaError_t r = cudaFuncSetAttribute(lin_bf16_kernel<1, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (r == cudaSuccess) r = cudaFuncSetAttribute(lin_bf16_kernel<2, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (r == cudaSuccess) r = cudaFuncSetAttribute(lin_bf16_kernel<1, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (r == cudaSuccess) r = cudaFuncSetAttribute(lin_bf16_kernel<2, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (r == cudaSuccess) r = cudaFuncSetAttribute(lin_bf16_kernel<2, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (r == cudaSuccess) r = cudaFuncSetAttribute(lin_bf16_kernel<1, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
    if (r != cudaSuccess) return static_cast<int>(r);
    ready[dev] = true;
  }
  const bool pair = p->mtiles == 2 && p->splits == 1 && p->nt == 128 && (grouped || (p->M_pad / 128) % 2 == 0);
  if (grouped && p->mtiles == 2 && !pair) return static_cast<int>(cudaErrorInvalidValue);      // (the table's tiles would not fit)
  const int abytes = p->nt * 128 * (pair ? 2 : 1);
  int stages = (kSmem - 1024) / (static_cast<int>(kLinTile) + abytes);
  if (stages > kLinMaxStages) stages = kLinMaxStages;
  const int smem = stages * (static_cast<int>(kLinTile) + abytes) + 1024;      // (at least 3 stages: a staged tile of 128 rows fits)
  const int tiles_m = pair ? (p->M + 255) / 256 : (p->M + p->nt - 1) / p->nt;
  const dim3 grid(tiles_m, p->N_pad / 256, p->splits);
  const dim3 ggrid(grouped ? p->group_max : 1, p->N_pad / 256, 1);
  auto go = [&](auto kernel, const dim3& g) { return launch(kernel, g, dim3(kLinThreads), smem, stream, 2, q, stages); };
  cudaError_t r;
  if (grouped && p->src_row) r = pair ? go(lin_bf16_kernel<2, 2>, ggrid) : go(lin_bf16_kernel<1, 2>, ggrid);
  else if (grouped) r = pair ? go(lin_bf16_kernel<2, 1>, ggrid) : go(lin_bf16_kernel<1, 1>, ggrid);
  else r = pair ? go(lin_bf16_kernel<2, 0>, grid) : go(lin_bf16_kernel<1, 0>, grid);
  if (r != cudaSuccess || p->fuse) return static_cast<int>(r);
  return static_cast<int>(launch(lin_epi_kernel, dim3(p->M), dim3(256), 0, stream, 0, *p));
}

extern "C" int saber_stream_embed_launch(const saber::StreamEmbedParams* p, cudaStream_t stream) {
  if (p->M <= 0) return static_cast<int>(cudaErrorInvalidValue);
  return static_cast<int>(saber::launch(saber::stream_embed_kernel, dim3(p->M), dim3(256), 0, stream, 0, *p));
}

extern "C" int saber_stream_norm_launch(const saber::StreamNormParams* p, cudaStream_t stream) {
  if (p->n <= 0) return static_cast<int>(cudaErrorInvalidValue);
  return static_cast<int>(saber::launch(saber::stream_norm_kernel, dim3(p->n), dim3(256), 0, stream, 0, *p));
}
