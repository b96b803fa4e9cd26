// Grouped-query attention over tiled pages.
//
//   conv     where q, k and v pass a convolution: the convolved rows with the weights of q and k, their sums of squares, normed
//            values; the kernels behind it read these rows instead of the projections
//   append   keys (normed) and values of this step's rows into their pages; for the tcgen05 form also the queries
//   form 2   flash_tc.cu: prompt portions
//   form 1   decoding and short portions: the query heads of a key head are the rows of an `mma.sync` tile, pages arrive
//            by bulk copies, keys are split over CTAs and the last CTA of a row to finish merges the parts.  A step
//            with one row per sequence appends its own key and value, so that it is the only launch.
//   form 0   a CTA per (row, head) on the CUDA cores: fp32 models and sizes the other forms do not take
#include "flash_tc.h"
#include "gqa.h"
#include "launch.cuh"
#include "mla_device.cuh"
#include "rotary.cuh"

namespace saber {

constexpr float kGqaLog2e = 1.4426950408889634f;
constexpr int kPage = 64;

// element of a page's key / value head block
__device__ __forceinline__ int bf16_key_at(int key, int d) { return (d >> 6) * 4096 + key * 64 + (((((d & 63) >> 3) ^ key) & 7) << 3) + (d & 7); }
__device__ __forceinline__ int bf16_val_at(int KP, int key, int v) { return kPage * KP + v * 64 + ((((key >> 3) ^ v) & 7) << 3) + (key & 7); }
template <typename T> struct Page;
template <> struct Page<__nv_bfloat16> {
  static __device__ __forceinline__ int key(const GqaParams&, int t, int d) { return bf16_key_at(t, d); }
  static __device__ __forceinline__ int val(const GqaParams& p, int t, int v) { return bf16_val_at(p.KP, t, v); }
  static __device__ __forceinline__ float load(const void* b, size_t i) { return __bfloat162float(static_cast<const __nv_bfloat16*>(b)[i]); }
  static __device__ __forceinline__ void store(void* b, size_t i, float x) { static_cast<__nv_bfloat16*>(b)[i] = __float2bfloat16(x); }
};
template <> struct Page<float> {
  static __device__ __forceinline__ int key(const GqaParams& p, int t, int d) { return t * p.KP + d; }
  static __device__ __forceinline__ int val(const GqaParams& p, int t, int v) { return kPage * p.KP + t * p.VP + v; }
  static __device__ __forceinline__ float load(const void* b, size_t i) { return static_cast<const float*>(b)[i]; }
  static __device__ __forceinline__ void store(void* b, size_t i, float x) { static_cast<float*>(b)[i] = x; }
};
__device__ __forceinline__ size_t page_block(const GqaParams& p, int page, int g) {
  return (static_cast<size_t>(page) * p.G + g) * kPage * (p.KP + p.VP);
}
// reciprocal root mean square of row m's queries (isk: keys) over all heads, by a warp
constexpr int kConvPart = 256;            // columns of a partial sum
__host__ __device__ constexpr int conv_parts(int n) { return (n + kConvPart - 1) / kConvPart; }
__device__ __forceinline__ float row_scale(const GqaParams& p, int m, int isk, int lane) {
  const int pq = conv_parts(p.H * p.D), pk = conv_parts(p.G * p.D);
  const float* ss = p.row_ss + static_cast<size_t>(m) * (pq + pk) + (isk ? pq : 0);
  float s = 0.f;
  for (int i = lane; i < (isk ? pk : pq); i += 32) s += ss[i];
  return 1.f / sqrtf(mla_warp_sum(s) / static_cast<float>((isk ? p.G : p.H) * p.D) + p.eps);
}
// reciprocal root mean square of the D values of a head of row m (a warp), 1 without the norm
__device__ __forceinline__ float head_scale(const GqaParams& p, const float* x, int m, int isk, int lane) {
  if (p.taps > 0) return row_scale(p, m, isk, lane);
  if (!p.qk_norm) return 1.f;
  float sq = 0.f;
  for (int d = lane; d < p.D; d += 32) sq = fmaf(x[d], x[d], sq);
  return 1.f / sqrtf(mla_warp_sum(sq) / static_cast<float>(p.D) + p.eps);
}

__device__ __forceinline__ float gated(const GqaParams& p, int m, int h, int v, float y) {
  y *= p.out_scale;
  if (p.gate == nullptr) return y;
  return y / (1.f + expf(-p.gate[static_cast<size_t>(m) * p.ld_gate + h * p.V + v]));
}

// slot of a sequence (< 0: none)
__device__ __forceinline__ int gqa_slot(const GqaParams& p, int j) {
  const int s = p.slots[j];
  if (s >= p.n_slots) {
    if (p.err) atomicCAS(p.err, 0u, static_cast<uint32_t>(kErrBadIndex));
    return -1;
  }
  return s;
}
struct ConvChannels {                             // q | k | v
  int nq, nk, nv;
  __device__ __forceinline__ explicit ConvChannels(const GqaParams& p) : nq(p.H * p.D), nk(p.G * p.D), nv(p.G * p.V) {}
  __device__ __forceinline__ int all() const { return nq + nk + nv; }
  __device__ __forceinline__ int column(const GqaParams& p, int c) const { return c < nq ? p.rq_off + c : c < nq + nk ? p.rk_off + c - nq : p.rv_off + c - nq - nk; }
};

// The last rows of sequence j become the ring's (they are the inputs of the next portion's first convolutions).
__device__ __forceinline__ void conv_ring(const GqaParams& p, int j) {
  const int r0 = p.cu_rows[j], n = p.cu_rows[j + 1] - r0, slot = n > 0 ? gqa_slot(p, j) : -1;
  if (slot < 0) return;
  const ConvChannels ch(p);
  float* hist = p.hist + static_cast<size_t>(slot) * p.taps * ch.all();
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < ch.all(); c += gridDim.y * blockDim.x)
    for (int t = max(0, n - p.taps); t < n; ++t)
      hist[static_cast<size_t>(p.pos[r0 + t] % p.taps) * ch.all() + c] = p.raw[static_cast<size_t>(r0 + t) * p.ld_raw + ch.column(p, c)];
}

constexpr int kConvRows = 8;              // rows of a strip

template <int VEC> struct ConvVec;
template <> struct ConvVec<4> { typedef float4 T; };
template <> struct ConvVec<1> { typedef float T; };
__device__ __forceinline__ float4 conv_fma(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
__device__ __forceinline__ float conv_fma(float a, float b, float c) { return fmaf(a, b, c); }
__device__ __forceinline__ float conv_dot(float4 a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }
__device__ __forceinline__ float conv_dot(float a) { return a * a; }
__device__ __forceinline__ float4 conv_mul(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float conv_mul(float a, float b) { return a * b; }
__device__ __forceinline__ float4 conv_scale(float4 a, float s) { return make_float4(a.x * s, a.y * s, a.z * s, a.w * s); }
__device__ __forceinline__ float conv_scale(float a, float s) { return a * s; }

// Up to kConvRows neighbouring rows of one sequence: the first is row m (its t-th of this step, at position pos).
struct ConvRun {
  int m, n, t, pos;
  float* hist;                            // of the slot, or null
};
// Channels c .. c + VEC - 1 (column col of the rows) of a run, convolved.  TAPS: their number when known at compile time, else 0.
template <int VEC, int TAPS, int ROWS>
__device__ __forceinline__ void conv_run(const GqaParams& p, const ConvRun& run, int C, int c, int col, typename ConvVec<VEC>::T (&y)[ROWS]) {
  typedef typename ConvVec<VEC>::T V;
  const float* x = p.raw + static_cast<size_t>(run.m) * p.ld_raw + col;
  const float* w = p.conv_w + c;
  auto input = [&](int i) -> V {          // of row m + i, earlier ones from the ring
    if (run.t + i >= 0) return *reinterpret_cast<const V*>(x + static_cast<ptrdiff_t>(i) * p.ld_raw);
    if (run.pos + i >= 0 && run.hist != nullptr) return *reinterpret_cast<const V*>(run.hist + static_cast<size_t>((run.pos + i) % p.taps) * C + c);
    return V{};
  };
#pragma unroll
  for (int r = 0; r < ROWS; ++r) y[r] = V{};
  if constexpr (TAPS > 0) {
    V u[TAPS - 1 + ROWS], f[TAPS];
#pragma unroll
    for (int i = 0; i < TAPS; ++i) f[i] = *reinterpret_cast<const V*>(w + static_cast<size_t>(i) * C);
#pragma unroll
    for (int i = 0; i < TAPS - 1 + ROWS; ++i) u[i] = i - (TAPS - 1) < run.n ? input(i - (TAPS - 1)) : V{};
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
#pragma unroll
      for (int i = 0; i < TAPS; ++i) y[r] = conv_fma(u[r + i], f[i], y[r]);
  } else {
    for (int i = 0; i < p.taps; ++i) {
      const V f = *reinterpret_cast<const V*>(w + static_cast<size_t>(i) * C);
#pragma unroll
      for (int r = 0; r < ROWS; ++r)
        if (r < run.n) y[r] = conv_fma(input(r - (p.taps - 1) + i), f, y[r]);
    }
  }
  if (p.max_rows == 1 && run.hist != nullptr)                      // (no token of this step reads that row)
    *reinterpret_cast<V*>(run.hist + static_cast<size_t>(run.pos % p.taps) * C + c) = input(0);
}

// grid (ceil(M / ROWS), ceil(items / 4)), 128 threads; a warp per strip of rows and item: 256 columns of q, then of k, then a value
// head.  Columns of cx from 0 = q, k_off = k, v_off = v on (as the kernels behind it read them).
template <int VEC, int TAPS, int ROWS>
__global__ void __launch_bounds__(128) gqa_conv_kernel(const __grid_constant__ GqaParams p) {
  pdl_trigger();
  pdl_wait();
  typedef typename ConvVec<VEC>::T V;
  const int lane = threadIdx.x & 31, item = blockIdx.y * 4 + (threadIdx.x >> 5);
  const ConvChannels ch(p);
  const int C = ch.all(), pq = conv_parts(ch.nq), pk = conv_parts(ch.nk);
  if (item >= pq + pk + p.G) return;
  const int end = min(p.M, (static_cast<int>(blockIdx.x) + 1) * ROWS);
  for (int m = blockIdx.x * ROWS; m < end;) {
    const int j = mla_seq_of_row(p.cu_rows, p.nseq, m);
    if (j < 0) return;                                              // (padding rows come last)
    const int slot = gqa_slot(p, j);
    const ConvRun run = {m, min(end, p.cu_rows[j + 1]) - m, m - p.cu_rows[j], p.pos[m], slot < 0 ? nullptr : p.hist + static_cast<size_t>(slot) * p.taps * C};
    m += run.n;
    float* o = p.cx + static_cast<size_t>(run.m) * p.ldc;
    float sq[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) sq[r] = 0.f;
    if (item < pq + pk) {
      const bool isk = item >= pq;
      const int first = (isk ? item - pq : item) * kConvPart, n = min(isk ? ch.nk : ch.nq, first + kConvPart);
      const float* w = isk ? p.k_w : p.q_w;
      for (int c = first + lane * VEC; c < n; c += 32 * VEC) {
        V y[ROWS];
        conv_run<VEC, TAPS, ROWS>(p, run, C, (isk ? ch.nq : 0) + c, (isk ? p.rk_off : p.rq_off) + c, y);
        const V f = *reinterpret_cast<const V*>(w + c);
        float* d = o + (isk ? p.k_off : p.q_off) + c;
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
          if (r < run.n) {
            sq[r] += conv_dot(y[r]);
            *reinterpret_cast<V*>(d + static_cast<size_t>(r) * p.ldc) = conv_mul(y[r], f);
          }
      }
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        sq[r] = mla_warp_sum(sq[r]);
        if (lane == 0 && r < run.n) p.row_ss[static_cast<size_t>(run.m + r) * (pq + pk) + item] = sq[r];
      }
    } else {
      const int g = item - pq - pk;
      float* d = o + p.v_off + g * p.V;
      for (int v = lane * VEC; v < p.V; v += 32 * VEC) {
        V y[ROWS];
        conv_run<VEC, TAPS, ROWS>(p, run, C, ch.nq + ch.nk + g * p.V + v, p.rv_off + g * p.V + v, y);
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
          if (r < run.n) {
            sq[r] += conv_dot(y[r]);
            *reinterpret_cast<V*>(d + static_cast<size_t>(r) * p.ldc + v) = y[r];
          }
      }
      if (!p.v_norm) continue;
#pragma unroll
      for (int r = 0; r < ROWS; ++r) sq[r] = 1.f / sqrtf(mla_warp_sum(sq[r]) / static_cast<float>(p.V) + p.eps);
      for (int v = lane * VEC; v < p.V; v += 32 * VEC)              // (a lane's own values)
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
          if (r < run.n) {
            V* a = reinterpret_cast<V*>(d + static_cast<size_t>(r) * p.ldc + v);
            *a = conv_scale(*a, sq[r]);
          }
    }
  }
}

template <int VEC, int TAPS>
static cudaError_t conv_rows_go(const GqaParams& p, cudaStream_t stream) {
  const int items = conv_parts(p.H * p.D) + conv_parts(p.G * p.D) + p.G;
  if (p.max_rows == 1) return launch(gqa_conv_kernel<VEC, TAPS, 1>, dim3(p.M, (items + 3) / 4), dim3(128), 0, stream, 2, p);
  return launch(gqa_conv_kernel<VEC, TAPS, kConvRows>, dim3((p.M + kConvRows - 1) / kConvRows, (items + 3) / 4), dim3(128), 0, stream, 2, p);
}
static cudaError_t conv_go(const GqaParams& p, cudaStream_t stream) {
  if (((p.H * p.D) & 3) || ((p.G * p.D) & 3) || (p.V & 3)) return conv_rows_go<1, 0>(p, stream);
  switch (p.taps) {
    case 2: return conv_rows_go<4, 2>(p, stream);
    case 3: return conv_rows_go<4, 3>(p, stream);
    case 4: return conv_rows_go<4, 4>(p, stream);
    default: return conv_rows_go<4, 0>(p, stream);
  }
}

// Four rows of a head from x on (scale: their reciprocal root mean squares where they are known; rows past n repeat the last), divided by their root mean square and rotated by the tables
// at t (rot floats a row); put(row, d, four values) takes the pieces.  D a multiple of 4, at most 256; rot a multiple of 8.
template <typename Put>
__device__ __forceinline__ void normed_rows4(const GqaParams& p, const float* x, int n, const float* scale, int lane, const float* t, const Put& put) {
  float4 v[4][2];
  float sq[4];
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int d = u * 128 + lane * 4;
      v[r][u] = d < p.D ? *reinterpret_cast<const float4*>(x + static_cast<size_t>(min(r, n - 1)) * p.ldx + d) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    if (!p.qk_norm || p.taps > 0) break;
    sq[r] = 0.f;
#pragma unroll
    for (int u = 0; u < 2; ++u) sq[r] += v[r][u].x * v[r][u].x + v[r][u].y * v[r][u].y + v[r][u].z * v[r][u].z + v[r][u].w * v[r][u].w;
  }
  if (p.qk_norm && p.taps == 0)
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int r = 0; r < 4; ++r) sq[r] += __shfl_xor_sync(0xffffffffu, sq[r], o);
  if (p.rot > 0) {                                // (the partner's four values: another lane's, read again)
    const int half = p.rot / 2;
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int d = u * 128 + lane * 4;
        if (d >= p.rot) continue;
        const bool lo = d < half;
        const float* tr = t + min(r, n - 1) * p.rot + (lo ? d : d - half);
        const float4 o4 = *reinterpret_cast<const float4*>(x + static_cast<size_t>(min(r, n - 1)) * p.ldx + (lo ? d + half : d - half));
        const float4 c = *reinterpret_cast<const float4*>(tr), s = *reinterpret_cast<const float4*>(tr + half);
        const float sg = lo ? -1.f : 1.f;
        float4& w = v[r][u];
        w = make_float4(w.x * c.x + sg * o4.x * s.x, w.y * c.y + sg * o4.y * s.y, w.z * c.z + sg * o4.z * s.z, w.w * c.w + sg * o4.w * s.w);
      }
  }
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    if (r >= n) break;
    const float s = p.taps > 0 ? scale[r] : p.qk_norm ? 1.f / sqrtf(sq[r] / static_cast<float>(p.D) + p.eps) : 1.f;
#pragma unroll
    for (int u = 0; u < 2; ++u) put(r, u * 128 + lane * 4, make_float4(v[r][u].x * s, v[r][u].y * s, v[r][u].z * s, v[r][u].w * s));
  }
}
__device__ __forceinline__ uint2 pack4(float4 v) { return make_uint2(pack2(v.x, v.y), pack2(v.z, v.w)); }

// grid (ceil(M / 8), ceil(items / 8)) and, behind a convolution, nseq more columns that update the rings; 256 threads; a warp per (head, eight rows): query heads (tcgen05 form only), then
// key heads, then value heads.  Eight values of neighbouring tokens leave as one 16-byte piece where a page allows it.
template <typename T>
__global__ void __launch_bounds__(256) gqa_append_kernel(const __grid_constant__ GqaParams p) {
  pdl_wait();
  extern __shared__ __align__(16) float rot_s[];  // rotation tables of the eight rows
  const int lane = threadIdx.x & 31;
  int item = blockIdx.y * 8 + (threadIdx.x >> 5);
  const int m0 = blockIdx.x * 8, n = min(8, p.M - m0);
  if (n <= 0) {
    conv_ring(p, static_cast<int>(blockIdx.x) - (p.M + 7) / 8);
    return;
  }
  const bool fast = sizeof(T) == 2 && (p.D & 3) == 0 && p.D <= 256 && (p.rot & 7) == 0;
  __shared__ float scale_s[2][8];                 // behind a convolution: of the rows' queries and keys
  if (p.rot > 0 || p.taps > 0) {
    for (int r = threadIdx.x >> 5; r < n; r += 8) {
      if (p.rot > 0) rotary_table(rot_s + r * p.rot, p.freq, p.rot, p.rot_amp, p.pos[m0 + r], lane, 32);
      if (p.taps > 0) {
        const float a = row_scale(p, m0 + r, 0, lane), b = row_scale(p, m0 + r, 1, lane);
        if (lane == 0) {
          scale_s[0][r] = a;
          scale_s[1][r] = b;
        }
      }
    }
    __syncthreads();
  }
  if (p.form == 2) {
    if (item < p.H) {
      __nv_bfloat16* q0 = static_cast<__nv_bfloat16*>(p.q) + (static_cast<size_t>(m0) * p.H + item) * p.DK;
      const float* x0 = p.x + static_cast<size_t>(m0) * p.ldx + p.q_off + item * p.D;
      if (fast) {
        for (int r0 = 0; r0 < n; r0 += 4)
          normed_rows4(p, x0 + static_cast<size_t>(r0) * p.ldx, n - r0, scale_s[0] + r0, lane, rot_s + r0 * p.rot, [&](int r, int d, float4 v) {
            if (d < p.DK) *reinterpret_cast<uint2*>(q0 + static_cast<size_t>(r0 + r) * p.H * p.DK + d) = pack4(v);      // (zeros from D on)
          });
        return;
      }
      for (int r = 0; r < n; ++r) {
        const float* x = x0 + static_cast<size_t>(r) * p.ldx;
        const float s = head_scale(p, x, m0 + r, 0, lane);
        for (int d = lane; d < p.DK; d += 32) q0[static_cast<size_t>(r) * p.H * p.DK + d] = __float2bfloat16(d < p.D ? rotary_half(x, d, rot_s + r * p.rot, p.rot) * s : 0.f);
      }
      return;
    }
    item -= p.H;
  }
  if (p.k_off < 0 || item >= 2 * p.G) return;
  const bool isv = item >= p.G;
  const int g = isv ? item - p.G : item;
  int slot[8];
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    slot[r] = r < n ? p.slot_map[m0 + r] : -1;
    if (slot[r] >= p.n_blocks * kPage) {
      if (lane == 0 && p.err) atomicCAS(p.err, 0u, static_cast<uint32_t>(kErrBadIndex));
      slot[r] = -1;
    }
  }
  if (!isv) {
    const float* x0 = p.x + static_cast<size_t>(m0) * p.ldx + p.k_off + g * p.D;
    if (fast) {
#pragma unroll
      for (int r0 = 0; r0 < 8; r0 += 4) {
        if (r0 >= n) break;
        normed_rows4(p, x0 + static_cast<size_t>(r0) * p.ldx, n - r0, scale_s[1] + r0, lane, rot_s + r0 * p.rot, [&](int r, int d, float4 v) {
          const int s = r == 0 ? slot[r0] : r == 1 ? slot[r0 + 1] : r == 2 ? slot[r0 + 2] : slot[r0 + 3];
          if (s >= 0 && d < p.D)
            *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p.cache) + page_block(p, s / kPage, g) + bf16_key_at(s % kPage, d)) = pack4(v);
        });
      }
      return;
    }
    for (int r = 0; r < n; ++r) {
      const int s = p.slot_map[m0 + r];
      if (s < 0 || s >= p.n_blocks * kPage) continue;
      const float* x = x0 + static_cast<size_t>(r) * p.ldx;
      const float sc = head_scale(p, x, m0 + r, 1, lane);
      const size_t b = page_block(p, s / kPage, g);
      for (int d = lane; d < p.D; d += 32) Page<T>::store(p.cache, b + Page<T>::key(p, s % kPage, d), rotary_half(x, d, rot_s + r * p.rot, p.rot) * sc);
    }
    return;
  }
  bool whole = sizeof(T) == 2 && slot[0] >= 0 && (slot[0] & 7) == 0;
#pragma unroll
  for (int r = 1; r < 8; ++r) whole = whole && slot[r] == slot[0] + r;
  const float* x = p.x + static_cast<size_t>(m0) * p.ldx + p.v_off + g * p.V;
  for (int v = lane; v < p.V; v += 32) {
    float y[8];
#pragma unroll
    for (int r = 0; r < 8; ++r) y[r] = slot[r] >= 0 ? x[static_cast<size_t>(r) * p.ldx + v] : 0.f;
    if (whole) {
      __nv_bfloat16* c = static_cast<__nv_bfloat16*>(p.cache) + page_block(p, slot[0] / kPage, g) + bf16_val_at(p.KP, slot[0] % kPage, v);
      *reinterpret_cast<uint4*>(c) = make_uint4(pack2(y[0], y[1]), pack2(y[2], y[3]), pack2(y[4], y[5]), pack2(y[6], y[7]));
    } else {
#pragma unroll
      for (int r = 0; r < 8; ++r)
        if (slot[r] >= 0) Page<T>::store(p.cache, page_block(p, slot[r] / kPage, g) + Page<T>::val(p, slot[r] % kPage, v), y[r]);
    }
  }
}

// grid (M, H), 128 threads: one query row of one head, 64 keys at a time
template <typename T>
__global__ void __launch_bounds__(128) gqa_row_kernel(const __grid_constant__ GqaParams p) {
  pdl_wait();
  extern __shared__ float sm[];                   // q [D] | scores [64] | output [V] | rotation table
  __shared__ float scale_s;
  const int m = blockIdx.x, h = blockIdx.y, g = h / (p.H / p.G);
  const int j = mla_seq_of_row(p.cu_rows, p.nseq, m);
  if (j < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* sc = sm + p.D;
  float* o = sc + kPage;
  const float* x = p.x + static_cast<size_t>(m) * p.ldx + p.q_off + h * p.D;
  float* rot_s = o + p.V;
  if (warp == 0) {
    const float s = head_scale(p, x, m, 0, lane);
    if (lane == 0) scale_s = s;
  }
  if (p.rot > 0) rotary_table(rot_s, p.freq, p.rot, p.rot_amp, p.pos[m], threadIdx.x, 128);
  __syncthreads();
  // (queries are rounded like the keys they meet)
  for (int d = threadIdx.x; d < p.D; d += 128) {
    const float q = rotary_half(x, d, rot_s, p.rot) * scale_s;
    sm[d] = sizeof(T) == 2 ? __bfloat162float(__float2bfloat16(q)) : q;
  }
  for (int v = threadIdx.x; v < p.V; v += 128) o[v] = 0.f;
  const int pos = p.pos[m], low = first_key(pos, p.chunk, p.window);
  float mx = -INFINITY, l = 0.f;
  for (int pg = low / kPage; pg <= pos / kPage; ++pg) {
    const size_t b = page_block(p, page_at(p, j, pg), g);
    const int t0 = max(0, low - pg * kPage), t1 = min(kPage, pos + 1 - pg * kPage);
    __syncthreads();
    for (int t = t0 + warp; t < t1; t += 4) {
      float s = 0.f;
      for (int d = lane; d < p.D; d += 32) s = fmaf(sm[d], Page<T>::load(p.cache, b + Page<T>::key(p, t, d)), s);
      s = mla_warp_sum(s) * p.scale;
      if (lane == 0) sc[t] = p.softcap > 0.f ? p.softcap * tanhf(s / p.softcap) : s;
    }
    __syncthreads();
    const float a = lane >= t0 && lane < t1 ? sc[lane] : -INFINITY, c = lane + 32 >= t0 && lane + 32 < t1 ? sc[lane + 32] : -INFINITY;
    const float mn = fmaxf(mx, mla_warp_max(fmaxf(a, c)));          // (every page of the walk has a visible key)
    const float ea = expf(a - mn), ec = expf(c - mn), corr = expf(mx - mn);
    l = l * corr + mla_warp_sum(ea + ec);
    mx = mn;
    __syncthreads();
    if (warp == 0) { sc[lane] = ea; sc[lane + 32] = ec; }
    __syncthreads();
    for (int v = threadIdx.x; v < p.V; v += 128) {
      float s = o[v] * corr;
      for (int t = t0; t < t1; ++t) s = fmaf(sc[t], Page<T>::load(p.cache, b + Page<T>::val(p, t, v)), s);
      o[v] = s;
    }
  }
  if (p.sink != nullptr) l += expf(p.sink[h] - mx);                 // (infinite: the sink takes everything)
  for (int v = threadIdx.x; v < p.V; v += 128) operand_store1(p.out, m, p.out_k0 + h * p.V + v, gated(p, m, h, v, o[v] / l));
}

// grid (M, G, splits), 128 threads.  MT: 16-row tiles of query heads.  NC: 8-column groups of a value per warp.
template <int MT, int NC>
__global__ void __launch_bounds__(128) gqa_split_kernel(const __grid_constant__ GqaParams p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ uint64_t bars[2];
  __shared__ float corr_s[MT * 16], l_s[MT * 16];
  __shared__ uint32_t last_s;
  const int m = blockIdx.x, g = blockIdx.y, sp = blockIdx.z;
  const int j = mla_seq_of_row(p.cu_rows, p.nseq, m);
  if (j < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, hq = p.H / p.G;
  const int pos = p.pos[m], low = first_key(pos, p.chunk, p.window);
  const int page0 = low / kPage, pages = pos / kPage + 1 - page0;
  const int per = (pages + p.splits - 1) / p.splits;
  const int pa = page0 + sp * per, n = min(per, page0 + pages - pa);       // this CTA's pages (n <= 0: none)
  const uint32_t stage = 128u * static_cast<uint32_t>(p.KP + p.VP);
  const uint32_t kv_s = (smem_u32(smem_raw) + 127u) & ~127u;
  const uint32_t qs = static_cast<uint32_t>(p.DK) * 2u + 16u;              // row stride: an odd number of 16-byte units
  const uint32_t q_s = kv_s + 2 * stage;
  const uint32_t p_s = q_s + MT * 16 * qs;                                 // probabilities, bf16 [MT * 16][64 + 8]
  uint8_t* const base = smem_raw + (kv_s - smem_u32(smem_raw));
  float* s_f = reinterpret_cast<float*>(base + 2 * stage + MT * 16 * qs + MT * 16 * 144);      // scores [MT * 16][64 + 4]
  const bool append = p.max_rows == 1 && p.k_off >= 0 && n > 0 && pa + n == page0 + pages;     // the new token's page is mine
  __nv_bfloat16* new_s = reinterpret_cast<__nv_bfloat16*>(s_f + MT * 16 * 68);                 // key [KP] | value [VP] of the new token
  float* rot_s = reinterpret_cast<float*>(new_s + p.KP + p.VP);                                // rotation table of the position
  const uint32_t bar = smem_u32(bars);
  const uint8_t* cache = static_cast<const uint8_t*>(p.cache);
  auto fetch = [&](int it) {
    mbar_arrive_expect_tx(bar + 8 * (it & 1), stage);
    bulk_g2s(kv_s + (it & 1) * stage, cache + page_block(p, page_at(p, j, pa + it), g) * 2, stage, bar + 8 * (it & 1));
  };
  int issued = 0;
  if (threadIdx.x == 0) {
    mbar_init(bar, 1);
    mbar_init(bar + 8, 1);
    mbar_init_fence();
    for (; issued < min(2, n); ++issued) fetch(issued);
  }
  const float* xr = p.x + static_cast<size_t>(m) * p.ldx;
  if (p.rot > 0) {
    rotary_table(rot_s, p.freq, p.rot, p.rot_amp, pos, threadIdx.x, 128);
    __syncthreads();
  }
  const float qs_all = p.taps > 0 ? row_scale(p, m, 0, lane) : 1.f;
  for (int r = warp; r < MT * 16; r += 4) {
    const float* x = xr + p.q_off + (g * hq + min(r, hq - 1)) * p.D;
    const float s = p.taps > 0 ? qs_all : head_scale(p, x, m, 0, lane);
    for (int d = lane * 2; d < p.DK; d += 64) {
      const float a = r < hq && d < p.D ? rotary_half(x, d, rot_s, p.rot) * s : 0.f, b = r < hq && d + 1 < p.D ? rotary_half(x, d + 1, rot_s, p.rot) * s : 0.f;
      asm volatile("st.shared.b32 [%0], %1;" ::"r"(q_s + r * qs + d * 2), "r"(pack2(a, b)) : "memory");
    }
  }
  for (int i = threadIdx.x; i < MT * 16 * 36; i += 128) asm volatile("st.shared.b32 [%0], %1;" ::"r"(p_s + i * 4), "r"(0) : "memory");
  if (threadIdx.x < MT * 16) corr_s[threadIdx.x] = 1.f;
  if (append) {
    const int slot = p.slot_map[m];
    const bool live = slot >= 0 && slot < p.n_blocks * kPage;
    __nv_bfloat16* c = static_cast<__nv_bfloat16*>(p.cache) + (live ? page_block(p, slot / kPage, g) : 0);
    if (warp == 0) {
      const float* x = xr + p.k_off + g * p.D;
      const float s = head_scale(p, x, m, 1, lane);
      for (int d = lane; d < p.D; d += 32) {
        new_s[d] = __float2bfloat16(rotary_half(x, d, rot_s, p.rot) * s);
        if (live) c[bf16_key_at(slot % kPage, d)] = new_s[d];
      }
    } else {
      for (int v = threadIdx.x - 32; v < p.V; v += 96) {
        new_s[p.KP + v] = __float2bfloat16(xr[p.v_off + g * p.V + v]);
        if (live) c[bf16_val_at(p.KP, slot % kPage, v)] = new_s[p.KP + v];
      }
    }
  }
  __syncthreads();
  const bool capped = p.softcap > 0.f;
  const float zs = capped ? 2.f * kGqaLog2e * p.scale / p.softcap : 0.f;
  float o[MT][NC][4] = {};
  float mx[4 * MT], l[4 * MT];                                      // rows warp, warp + 4, ... of the tile
#pragma unroll
  for (int i = 0; i < 4 * MT; ++i) { mx[i] = -INFINITY; l[i] = 0.f; }
  bool ok = true;
  int it = 0;
  for (; it < n; ++it) {
    const uint32_t kt = kv_s + (it & 1) * stage, vt = kt + kPage * 2 * p.KP;
    ok = __syncthreads_and(mbar_wait(bar + 8 * (it & 1), (it >> 1) & 1, p.err, kErrWaitFull)) != 0;
    if (!ok) break;
    if (append && it == n - 1) {
      __nv_bfloat16* c = reinterpret_cast<__nv_bfloat16*>(base + (it & 1) * stage);
      for (int d = threadIdx.x; d < p.D; d += 128) c[bf16_key_at(pos % kPage, d)] = new_s[d];
      for (int v = threadIdx.x; v < p.V; v += 128) c[bf16_val_at(p.KP, pos % kPage, v)] = new_s[p.KP + v];
      __syncthreads();
    }
    // scores: 16 keys per warp
    {
      float s[MT][2][4] = {};
      const uint32_t a_row = q_s + (lane & 15) * qs + ((lane >> 4) << 4);
      const int key = warp * 16 + ((lane >> 4) << 3) + (lane & 7);
      for (int st = 0; st < p.DK / 16; ++st) {
        const int c = st * 2 + ((lane >> 3) & 1);
        uint32_t b[4];
        ldsm4(b, kt + (c >> 3) * 8192 + key * 128 + (((c ^ key) & 7) << 4));
#pragma unroll
        for (int t = 0; t < MT; ++t) {
          uint32_t a[4];
          ldsm4(a, a_row + t * 16 * qs + st * 32);
          mma16816(s[t][0], a, b[0], b[1]);
          mma16816(s[t][1], a, b[2], b[3]);
        }
      }
      const int r = lane >> 2;
#pragma unroll
      for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int c = warp * 16 + i * 8 + (lane & 3) * 2;
          *reinterpret_cast<float2*>(s_f + (t * 16 + r) * 68 + c) = make_float2(s[t][i][0], s[t][i][1]);
          *reinterpret_cast<float2*>(s_f + (t * 16 + r + 8) * 68 + c) = make_float2(s[t][i][2], s[t][i][3]);
        }
    }
    __syncthreads();
    // running softmax
    const int key0 = (pa + it) * kPage + lane * 2;
#pragma unroll
    for (int i = 0; i < 4 * MT; ++i) {
      const int r = warp + 4 * i;
      if (r >= hq) continue;
      const float2 v = *reinterpret_cast<const float2*>(s_f + r * 68 + lane * 2);
      float a = v.x * p.scale, b = v.y * p.scale;
      if (capped) {
        a = p.softcap - __fdividef(2.f * p.softcap, 1.f + ex2(v.x * zs));
        b = p.softcap - __fdividef(2.f * p.softcap, 1.f + ex2(v.y * zs));
      }
      if (key0 < low || key0 > pos) a = -INFINITY;
      if (key0 + 1 < low || key0 + 1 > pos) b = -INFINITY;
      const float mn = fmaxf(mx[i], mla_warp_max(fmaxf(a, b)));     // (every page of the walk has a visible key)
      const float ea = ex2((a - mn) * kGqaLog2e), eb = ex2((b - mn) * kGqaLog2e), corr = ex2((mx[i] - mn) * kGqaLog2e);
      l[i] = l[i] * corr + mla_warp_sum(ea + eb);
      mx[i] = mn;
      asm volatile("st.shared.b32 [%0], %1;" ::"r"(p_s + r * 144 + lane * 4), "r"(pack2(ea, eb)) : "memory");
      if (lane == 0) corr_s[r] = corr;
    }
    __syncthreads();
    // values: this warp's columns
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      const float c0 = corr_s[t * 16 + (lane >> 2)], c1 = corr_s[t * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int i = 0; i < NC; ++i) { o[t][i][0] *= c0; o[t][i][1] *= c0; o[t][i][2] *= c1; o[t][i][3] *= c1; }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {                          // 32 keys
      uint32_t a[MT][2][4];
#pragma unroll
      for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int k = 0; k < 2; ++k) ldsm4(a[t][k], p_s + (t * 16 + (lane & 15)) * 144 + (half * 2 + k) * 32 + ((lane >> 4) << 4));
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int col = (warp * NC + i) * 8;
        if (col >= p.VP) break;
        const int v = col + (lane & 7), c = half * 4 + (lane >> 3);
        uint32_t b[4];
        ldsm4(b, vt + v * 128 + (((c ^ v) & 7) << 4));
#pragma unroll
        for (int t = 0; t < MT; ++t) {
          mma16816(o[t][i], a[t][0], b[0], b[1]);
          mma16816(o[t][i], a[t][1], b[2], b[3]);
        }
      }
    }
    __syncthreads();
    if (threadIdx.x == 0 && it + 2 < n) { fetch(it + 2); ++issued; }
  }
  if (!ok && threadIdx.x == 0)                                      // do not leave while an own copy is in flight
    for (int i = it; i < issued; ++i) mbar_wait(bar + 8 * (i & 1), (i >> 1) & 1, p.err, kErrWaitDrain);
#pragma unroll
  for (int i = 0; i < 4 * MT; ++i) {
    const int r = warp + 4 * i;
    if (r >= hq || lane != 0) continue;
    l_s[r] = p.sink != nullptr ? l[i] + ex2((p.sink[g * hq + r] - mx[i]) * kGqaLog2e) : l[i];    // (infinite: the sink takes everything)
    if (p.splits > 1) {
      float* d = p.ml + ((static_cast<size_t>(m) * p.H + g * hq + r) * p.splits + sp) * 2;
      __stcg(d, mx[i]);
      __stcg(d + 1, l[i]);
    }
  }
  __syncthreads();
#pragma unroll
  for (int t = 0; t < MT; ++t)
#pragma unroll
    for (int e2 = 0; e2 < 2; ++e2) {
      const int r = t * 16 + (lane >> 2) + e2 * 8;
      if (r >= hq) continue;
      const int h = g * hq + r;
      const float inv = 1.f / l_s[r];
      float* d = p.splits > 1 ? p.o_part + ((static_cast<size_t>(m) * p.H + h) * p.splits + sp) * p.VP : nullptr;
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int v = (warp * NC + i) * 8 + (lane & 3) * 2;
        if (v >= p.VP) break;
        const float a = o[t][i][e2 * 2], b = o[t][i][e2 * 2 + 1];
        if (d != nullptr) {
          if (n > 0) __stcg(reinterpret_cast<float2*>(d + v), make_float2(a, b));
        } else {
          if (v < p.V) operand_store1(p.out, m, p.out_k0 + h * p.V + v, gated(p, m, h, v, a * inv));
          if (v + 1 < p.V) operand_store1(p.out, m, p.out_k0 + h * p.V + v + 1, gated(p, m, h, v + 1, b * inv));
        }
      }
    }
  if (p.splits == 1) return;
  // the last part of the row to arrive merges them, in order
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    uint32_t* c = p.counters + static_cast<size_t>(m) * p.G + g;
    const bool last = atomicAdd(c, 1u) == static_cast<uint32_t>(p.splits) - 1u;
    if (last) *c = 0u;
    __threadfence();
    last_s = last ? 1u : 0u;
  }
  __syncthreads();
  if (!last_s) return;
  const float* ml = p.ml + (static_cast<size_t>(m) * p.H + g * hq) * p.splits * 2;
  for (int r = warp; r < hq; r += 4) {                              // weights of the parts (splits <= 32: a lane each)
    const float pm = lane < p.splits ? __ldcg(ml + (r * p.splits + lane) * 2) : -INFINITY;
    const float pl = lane < p.splits ? __ldcg(ml + (r * p.splits + lane) * 2 + 1) : 0.f;
    const float mm = mla_warp_max(pm);
    const float w = pm > -INFINITY ? ex2((pm - mm) * kGqaLog2e) : 0.f;
    const float tot = mla_warp_sum(w * pl) + (p.sink != nullptr ? ex2((p.sink[g * hq + r] - mm) * kGqaLog2e) : 0.f);
    s_f[r * 33 + lane] = w / tot;
  }
  __syncthreads();
  const float* part = p.o_part + (static_cast<size_t>(m) * p.H + g * hq) * p.splits * p.VP;
  for (int i = threadIdx.x; i < hq * p.V; i += 128) {
    const int r = i / p.V, v = i - r * p.V;
    float y = 0.f;
#pragma unroll 4
    for (int s = 0; s < p.splits; ++s) {
      const float w = s_f[r * 33 + s];
      if (w > 0.f) y = fmaf(w, __ldcg(part + (static_cast<size_t>(r) * p.splits + s) * p.VP + v), y);
    }
    operand_store1(p.out, m, p.out_k0 + (g * hq + r) * p.V + v, gated(p, m, g * hq + r, v, y));
  }
}

static int split_tiles(const GqaParams& p) {
  const int hq = p.H / p.G;
  return hq <= 16 ? 1 : hq <= 32 ? 2 : 4;
}
static int split_smem(const GqaParams& p) {
  const int rows = split_tiles(p) * 16;
  return 2 * 128 * (p.KP + p.VP) + rows * (p.DK * 2 + 16 + 144 + 68 * 4) + 2 * (p.KP + p.VP) + p.rot * 4 + 128;
}
template <int MT, int NC>
static int split_go(const GqaParams& p, cudaStream_t stream) {
  static bool ready[64];
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return static_cast<int>(cudaErrorInvalidDevice);
  if (!ready[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(gqa_split_kernel<MT, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    ready[dev] = true;
  }
  return static_cast<int>(launch(gqa_split_kernel<MT, NC>, dim3(p.M, p.G, p.splits), dim3(128), split_smem(p), stream, 2, p));
}
template <int NC>
static int split_mt(const GqaParams& p, cudaStream_t s) {
  const int mt = split_tiles(p);
  return mt == 1 ? split_go<1, NC>(p, s) : mt == 2 ? split_go<2, NC>(p, s) : split_go<4, NC>(p, s);
}

static int append_items(const GqaParams& p) {
  if (p.form == 1 && p.max_rows == 1) return 0;                     // the attention kernel appends by itself (the convolution kernel updates its rings)
  return (p.form == 2 ? p.H : 0) + (p.k_off >= 0 ? 2 * p.G : 0);
}

template <typename T>
static int gqa_go(GqaParams p, cudaStream_t stream) {
  p.gate = p.g_off < 0 ? nullptr : p.x + p.g_off;
  p.ld_gate = p.ldx;
  if (p.taps > 0) {
    p.raw = p.x;
    p.ld_raw = p.ldx;
    p.rq_off = p.q_off;
    p.rk_off = p.k_off;
    p.rv_off = p.v_off;
    p.x = p.cx;
    p.ldx = p.ldc;
    p.q_off = 0;
    p.k_off = (p.H * p.D + 7) & ~7;
    p.v_off = p.k_off + ((p.G * p.D + 7) & ~7);
    const cudaError_t e = conv_go(p, stream);
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  if (const int items = append_items(p)) {
    const int rings = p.taps > 0 && p.max_rows > 1 ? p.nseq : 0;
    const cudaError_t e = launch(gqa_append_kernel<T>, dim3((p.M + 7) / 8 + rings, (items + 7) / 8), dim3(256), 8 * p.rot * 4, stream, 0, p);
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  if (p.form == 0)
    return static_cast<int>(launch(gqa_row_kernel<T>, dim3(p.M, p.H), dim3(128), (p.D + kPage + p.V + p.rot) * 4, stream, 0, p));
  if (p.form == 1)
    return p.VP <= 32 ? split_mt<1>(p, stream) : p.VP <= 64 ? split_mt<2>(p, stream) : p.VP <= 128 ? split_mt<4>(p, stream) : split_mt<8>(p, stream);
  FlashParams f = {};
  f.q = p.q;
  f.k = p.cache;
  f.v = static_cast<const uint8_t*>(p.cache) + static_cast<size_t>(kPage) * p.KP * 2;
  f.k_stride = f.v_stride = static_cast<size_t>(kPage) * (p.KP + p.VP) * 2;
  f.cu_rows = p.cu_rows;
  f.kv_len = p.kv_len;
  f.block_table = p.block_table;
  f.out = p.out;
  f.out_k0 = p.out_k0;
  f.nseq = p.nseq;
  f.H = p.H;
  f.G = p.G;
  f.DK = p.DK;
  f.V = p.V;
  f.VP = p.VP;
  f.n_blocks = p.n_blocks;
  f.max_blocks = p.max_blocks;
  f.max_rows = p.max_rows;
  f.chunk = p.chunk;
  f.scale = p.scale;
  f.softcap = p.softcap;
  f.gate = p.gate;
  f.ldg = p.ld_gate;
  f.window = p.window;
  f.out_scale = p.out_scale;
  f.sink = p.sink;
  f.bound = p.qk_norm ? 1.02f * p.D : 0.f;        // (two vectors of root mean square one, and the rounding to bf16)
  f.err = p.err;
  return saber_flash_tc(&f, stream);
}

}  // namespace saber

extern "C" int saber_gqa_form(const saber::GqaParams* p) {
  if (p->f32 || p->page != saber::kPage || p->H / p->G > 64 || p->VP > 256 || (p->VP & 31) || (p->DK & 15) || (p->KP & 63) ||
      saber::split_smem(*p) > 224 * 1024)
    return 0;
  return saber_flash_tc_ok(p->page, p->DK, p->VP, p->scale, p->softcap) ? 2 : 1;
}

extern "C" int saber_gqa_launches(const saber::GqaParams* p) { return (p->taps > 0 ? 1 : 0) + (saber::append_items(*p) ? 2 : 1); }

extern "C" int saber_gqa_launch(const saber::GqaParams* p, cudaStream_t stream) {
  using namespace saber;
  if (p->M <= 0 || p->G <= 0 || p->H % p->G || p->page != kPage || p->D > p->DK || p->DK > p->KP || p->V > p->VP || p->cache == nullptr ||
      p->D > 2048 || p->V > 2048 || p->rot < 0 || (p->rot & 1) || p->rot > p->D || p->rot > 1024 || (p->rot > 0 && p->freq == nullptr) || p->form < 0 || p->form > saber_gqa_form(p) || (p->form == 2 && p->q == nullptr) ||
      (p->form == 1 && (p->splits < 1 || p->splits > 32 || (p->splits > 1 && (p->o_part == nullptr || p->ml == nullptr || p->counters == nullptr)))))
    return static_cast<int>(cudaErrorInvalidValue);
  if (p->window < 0 || (p->window > 0 && p->chunk > 0) ||
      (p->taps > 0 && (p->k_off < 0 || p->conv_w == nullptr || p->q_w == nullptr || p->k_w == nullptr || p->hist == nullptr || p->slots == nullptr ||
                       p->cx == nullptr || p->row_ss == nullptr || (p->ldc & 7) || p->ldc < ((p->H * p->D + 7) & ~7) + ((p->G * p->D + 7) & ~7) + p->G * p->V)))
    return static_cast<int>(cudaErrorInvalidValue);
  return p->f32 ? gqa_go<float>(*p, stream) : gqa_go<__nv_bfloat16>(*p, stream);
}
