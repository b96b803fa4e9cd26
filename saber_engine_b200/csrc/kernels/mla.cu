// Latent attention over a paged cache of latents.
//
// Absorbed form (decoding, short portions, fp32): the query is carried into the latent space, W_uk^T q, so that
// all heads of a row read the same cached row once; the weighted latents are carried out by W_uv.  Rows are
// independent (each knows its sequence and position), so any ragged batch is the same launch; keys may be
// split over CTAs and are merged by the output kernel.
#include "launch.cuh"
#include "mla_device.cuh"
#include "rotary.cuh"

namespace saber {

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// grid M, 256 threads: latent norm and rotated key into the cache, rotated query part (and, in the expanded
// form, the unrotated one) into q_eff
template <typename T>
__global__ void __launch_bounds__(256) mla_prep_kernel(const __grid_constant__ MlaParams p) {
  pdl_wait();
  __shared__ float red[8];
  extern __shared__ float rot[];                  // [R / 2] cosines, [R / 2] sines of this position
  const int m = blockIdx.x;
  if (mla_seq_of_row(p.cu_rows, p.nseq, m) < 0) return;
  const float* x = p.x + static_cast<size_t>(m) * p.ldx;
  const float* qx = p.q + static_cast<size_t>(m) * p.ldq + p.q_off;
  const int LD = p.CP + p.RP;
  const bool il = p.interleaved != 0;
  rotary_table(rot, p.freq, p.R, p.rot_amp, p.pos[m], threadIdx.x, 256);
  if (p.dkv_off >= 0) {
    const float* d = x + p.dkv_off;
    float sq = 0.f;
    for (int i = threadIdx.x; i < p.C; i += 256) sq += d[i] * d[i];
    sq = mla_warp_sum(sq);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
    __syncthreads();
    sq = 0.f;
    for (int w = 0; w < 8; ++w) sq += red[w];
    const float r = 1.f / sqrtf(sq / static_cast<float>(p.C) + p.eps);
    const int slot = p.slot_map[m];
    if (slot >= 0 && slot < p.n_blocks * p.page) {
      T* c = static_cast<T*>(p.cache) + static_cast<size_t>(slot) * LD;
      for (int i = threadIdx.x; i < p.CP; i += 256) c[i] = from_f<T>(i < p.C ? d[i] * r * p.dkv_norm[i] : 0.f);
      for (int i = threadIdx.x; i < p.RP; i += 256) c[p.CP + i] = from_f<T>(i < p.R ? rotary_value(d + p.C, i, rot, p.R, il) : 0.f);
    } else if (slot >= 0 && threadIdx.x == 0 && p.err) {
      atomicCAS(p.err, 0u, static_cast<uint32_t>(kErrBadIndex));
    }
  } else {
    __syncthreads();
  }
  const int KP = p.expand ? p.DP : p.CP;
  T* q = static_cast<T*>(p.q_eff) + static_cast<size_t>(m) * p.H * (KP + p.RP);
  for (int i = threadIdx.x; i < p.H * p.RP; i += 256) {
    const int h = i / p.RP, k = i - h * p.RP;
    q[static_cast<size_t>(h) * (KP + p.RP) + KP + k] = from_f<T>(k < p.R ? rotary_value(qx + h * (p.D + p.R) + p.D, k, rot, p.R, il) : 0.f);
  }
  if (p.expand)
    for (int i = threadIdx.x; i < p.H * p.DP; i += 256) {
      const int h = i / p.DP, k = i - h * p.DP;
      q[static_cast<size_t>(h) * (KP + p.RP) + k] = from_f<T>(k < p.D ? qx[h * (p.D + p.R) + k] : 0.f);
    }
}

// grid (ceil(CP / 128), H, ceil(M / 8)), 256 threads: q_eff[m][h][r] = sum_d W_uk[h D + d][r] q[m][h][d] for eight rows.
// 64 column pairs; four thread groups take a quarter of the d each and meet in shared memory.
template <typename T> struct Pair;
template <> struct Pair<float> {
  static __device__ __forceinline__ float2 load(const float* p) { return *reinterpret_cast<const float2*>(p); }
  static __device__ __forceinline__ void store(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
};
template <> struct Pair<__nv_bfloat16> {
  static __device__ __forceinline__ float2 load(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }
};

template <typename T>
__global__ void __launch_bounds__(256) mla_absorb_kernel(const __grid_constant__ MlaParams p) {
  pdl_wait();
  extern __shared__ float sm[];                   // q [D][8] | partial sums [3][64][16]
  float* part = sm + p.D * 8;
  const int h = blockIdx.y, mb = blockIdx.z * 8, rows = min(8, p.M - mb);
  for (int i = threadIdx.x; i < p.D * 8; i += 256) {
    const int r = i / p.D, d = i - r * p.D;
    sm[d * 8 + r] = r < rows ? p.q[static_cast<size_t>(mb + r) * p.ldq + p.q_off + h * (p.D + p.R) + d] : 0.f;
  }
  __syncthreads();
  const int cp = threadIdx.x & 63, quarter = threadIdx.x >> 6;
  const int c = blockIdx.x * 128 + cp * 2;         // CP is even
  const int per = (p.D + 3) / 4, d0 = quarter * per, d1 = min(p.D, d0 + per);
  float acc[8][2] = {};
  if (c < p.CP) {
    const T* w = static_cast<const T*>(p.w_uk) + static_cast<size_t>(h) * p.D * p.CP + c;
#pragma unroll 8
    for (int d = d0; d < d1; ++d) {
      const float2 wv = Pair<T>::load(w + static_cast<size_t>(d) * p.CP);
      const float4 a = *reinterpret_cast<const float4*>(sm + d * 8), b = *reinterpret_cast<const float4*>(sm + d * 8 + 4);
      const float q[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        acc[r][0] = fmaf(wv.x, q[r], acc[r][0]);
        acc[r][1] = fmaf(wv.y, q[r], acc[r][1]);
      }
    }
  }
  if (quarter > 0) {
#pragma unroll
    for (int r = 0; r < 8; ++r) *reinterpret_cast<float2*>(part + ((quarter - 1) * 8 + r) * 128 + cp * 2) = make_float2(acc[r][0], acc[r][1]);
  }
  __syncthreads();
  if (quarter > 0 || c >= p.CP) return;
  const int LD = p.CP + p.RP;
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    if (r >= rows) break;
#pragma unroll
    for (int g = 0; g < 3; ++g) {
      const float2 v = *reinterpret_cast<const float2*>(part + (g * 8 + r) * 128 + cp * 2);
      acc[r][0] += v.x;
      acc[r][1] += v.y;
    }
    Pair<T>::store(static_cast<T*>(p.q_eff) + (static_cast<size_t>(mb + r) * p.H + h) * LD + c, acc[r][0], acc[r][1]);
  }
}

// grid (M, H, splits), 128 threads: one query row of one head over its share of the keys, 64 at a time
constexpr int kRowKeys = 64, kRowMaxC = 8;         // latents of up to 1024 values

template <typename T>
__global__ void __launch_bounds__(128) mla_row_attn_kernel(const __grid_constant__ MlaParams p) {
  pdl_wait();
  extern __shared__ float sm[];                   // q [CP + RP] | scores [64]
  __shared__ const T* rows_s[kRowKeys];
  const int m = blockIdx.x, h = blockIdx.y, sp = blockIdx.z;
  const int j = mla_seq_of_row(p.cu_rows, p.nseq, m);
  if (j < 0) return;
  const int LD = p.CP + p.RP, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* sc = sm + LD;
  const T* q = static_cast<const T*>(p.q_eff) + (static_cast<size_t>(m) * p.H + h) * LD;
  for (int i = threadIdx.x; i < LD; i += 128) sm[i] = to_f<T>(q[i]);
  const int keys = p.pos[m] + 1;
  const int per = ((keys + p.splits - 1) / p.splits + kRowKeys - 1) / kRowKeys * kRowKeys;
  const int k0 = sp * per, k1 = min(keys, k0 + per);
  float acc[kRowMaxC] = {}, mx = -INFINITY, l = 0.f;
  for (int kb = k0; kb < k1; kb += kRowKeys) {
    const int n = min(kRowKeys, k1 - kb);
    __syncthreads();
    if (threadIdx.x < n) {
      const int key = kb + threadIdx.x;
      rows_s[threadIdx.x] = static_cast<const T*>(p.cache) + (static_cast<size_t>(page_at(p, j, key / p.page)) * p.page + key % p.page) * LD;
    }
    __syncthreads();
    for (int k = warp; k < n; k += 4) {
      const T* c = rows_s[k];
      float s = 0.f;
      for (int i = lane; i < LD; i += 32) s = fmaf(sm[i], to_f<T>(c[i]), s);
      s = mla_warp_sum(s);
      if (lane == 0) sc[k] = s * p.scale;
    }
    __syncthreads();
    const float a = lane < n ? sc[lane] : -INFINITY, b = lane + 32 < n ? sc[lane + 32] : -INFINITY;
    const float mn = fmaxf(mx, mla_warp_max(fmaxf(a, b)));
    const float ea = lane < n ? expf(a - mn) : 0.f, eb = lane + 32 < n ? expf(b - mn) : 0.f;
    const float corr = expf(mx - mn);
    l = l * corr + mla_warp_sum(ea + eb);
    mx = mn;
    __syncthreads();
    if (warp == 0) { sc[lane] = ea; sc[lane + 32] = eb; }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kRowMaxC; ++i) {
      const int c = i * 128 + threadIdx.x;
      if (c >= p.CP) break;
      float s = acc[i] * corr;
      for (int k = 0; k < n; ++k) s = fmaf(sc[k], to_f<T>(rows_s[k][c]), s);
      acc[i] = s;
    }
  }
  const size_t row = (static_cast<size_t>(m) * p.H + h) * p.splits + sp;
#pragma unroll
  for (int i = 0; i < kRowMaxC; ++i) {
    const int c = i * 128 + threadIdx.x;
    if (c < p.CP) p.o_part[row * p.CP + c] = acc[i];
  }
  if (threadIdx.x == 0) { p.ml[row * 2] = mx; p.ml[row * 2 + 1] = l; }
}

// grid (M, H), 128 threads: merges the key splits of a row's head into split 0's place, divided by the sum
__global__ void __launch_bounds__(128) mla_merge_kernel(const __grid_constant__ MlaParams p) {
  pdl_wait();
  __shared__ float wt[64];
  const int m = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31;
  if (mla_seq_of_row(p.cu_rows, p.nseq, m) < 0) return;
  const size_t row = (static_cast<size_t>(m) * p.H + h) * p.splits;
  if (threadIdx.x < 32) {
    const float* ml = p.ml + row * 2;
    float mx = -INFINITY, l = 0.f;
    for (int s = lane; s < p.splits; s += 32) mx = fmaxf(mx, ml[s * 2]);
    mx = mla_warp_max(mx);
    for (int s = lane; s < p.splits; s += 32) l += ml[s * 2] > -INFINITY ? ml[s * 2 + 1] * expf(ml[s * 2] - mx) : 0.f;
    l = mla_warp_sum(l);
    for (int s = lane; s < p.splits; s += 32) wt[s] = ml[s * 2] > -INFINITY ? expf(ml[s * 2] - mx) / l : 0.f;
  }
  __syncthreads();
  float* o = p.o_part + row * p.CP;
  for (int c = threadIdx.x * 4; c < p.CP; c += 512) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 6
    for (int s = 0; s < p.splits; ++s) {
      const float4 a = __ldcg(reinterpret_cast<const float4*>(o + static_cast<size_t>(s) * p.CP + c));
      const float w = wt[s];
      v.x = fmaf(a.x, w, v.x); v.y = fmaf(a.y, w, v.y); v.z = fmaf(a.z, w, v.z); v.w = fmaf(a.w, w, v.w);
    }
    *reinterpret_cast<float4*>(o + c) = v;         // read by this thread alone
  }
}

// grid (ceil(M / 8), H, ceil(V / 16)), 256 threads: the latents of eight rows through W_uv (a weight row is read once
// for the eight), gated
template <typename T>
__global__ void __launch_bounds__(256) mla_out_kernel(const __grid_constant__ MlaParams p) {
  pdl_wait();
  extern __shared__ float sm[];                   // [8][CP]
  const int mb = blockIdx.x * 8, h = blockIdx.y, rows = min(8, p.M - mb);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x * 4; i < 8 * p.CP; i += 1024) {
    const int r = i / p.CP, c = i - r * p.CP;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (r < rows && mla_seq_of_row(p.cu_rows, p.nseq, mb + r) >= 0)
      v = *reinterpret_cast<const float4*>(p.o_part + (static_cast<size_t>(mb + r) * p.H + h) * p.splits * p.CP + c);
    *reinterpret_cast<float4*>(sm + i) = v;
  }
  __syncthreads();
  const int v1 = min(p.V, static_cast<int>(blockIdx.z) * 16 + 16);
  for (int v = blockIdx.z * 16 + warp; v < v1; v += 8) {
    const T* w = static_cast<const T*>(p.w_uv) + (static_cast<size_t>(h) * p.V + v) * p.CP;
    float s[8] = {};
#pragma unroll 8
    for (int c = lane * 2; c < p.CP; c += 64) {
      const float2 wv = Pair<T>::load(w + c);
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        const float2 o = *reinterpret_cast<const float2*>(sm + r * p.CP + c);
        s[r] = fmaf(wv.x, o.x, s[r]);
        s[r] = fmaf(wv.y, o.y, s[r]);
      }
    }
#pragma unroll
    for (int r = 0; r < 8; ++r) s[r] = mla_warp_sum(s[r]);
    if (lane < rows) {
      float y = s[0];
#pragma unroll
      for (int r = 1; r < 8; ++r) y = lane == r ? s[r] : y;
      const float g = mla_gate(p, mb + lane, h, v);
      operand_store1(p.out, mb + lane, p.out_k0 + h * p.V + v, y / (1.f + expf(-g)));
    }
  }
}

template <typename T>
static int mla_go(const MlaParams& p, cudaStream_t stream) {
  cudaError_t e = launch(mla_prep_kernel<T>, dim3(p.M), dim3(256), p.R * 4 + 16, stream, 0, p);
  if (e != cudaSuccess) return static_cast<int>(e);
  if (p.expand) return saber_mla_expand_attn(&p, stream);
  e = launch(mla_absorb_kernel<T>, dim3((p.CP + 127) / 128, p.H, (p.M + 7) / 8), dim3(256), (p.D * 8 + 3 * 8 * 128) * 4, stream, 0, p);
  if (e != cudaSuccess) return static_cast<int>(e);
  if (saber_mla_decode_ok(&p)) {
    const int r = saber_mla_decode_attn(&p, stream);
    if (r != 0) return r;
  } else {
    e = launch(mla_row_attn_kernel<T>, dim3(p.M, p.H, p.splits), dim3(128), (p.CP + p.RP + kRowKeys) * 4, stream, 0, p);
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  e = launch(mla_merge_kernel, dim3(p.M, p.H), dim3(128), 0, stream, 0, p);
  if (e != cudaSuccess) return static_cast<int>(e);
  return static_cast<int>(launch(mla_out_kernel<T>, dim3((p.M + 7) / 8, p.H, (p.V + 15) / 16), dim3(256), 8 * p.CP * 4, stream, 0, p));
}

}  // namespace saber

extern "C" int saber_mla_launches(const saber::MlaParams* p) { return p->expand ? 3 : 5; }

extern "C" int saber_mla_launch(const saber::MlaParams* p, cudaStream_t stream) {
  using namespace saber;
  if (p->M <= 0 || p->C > p->CP || p->R > p->RP || (p->R & 1) || p->CP > 128 * kRowMaxC || p->D > 1024 || p->splits < 1 || p->splits > 64 ||
      p->q_eff == nullptr || p->cache == nullptr || p->q == nullptr)
    return static_cast<int>(cudaErrorInvalidValue);
  if (p->expand ? (p->k_exp == nullptr || p->v_exp == nullptr || saber_mla_expand_ok(p) < p->expand) : (p->o_part == nullptr || p->ml == nullptr))
    return static_cast<int>(cudaErrorInvalidValue);
  return p->f32 ? mla_go<float>(*p, stream) : mla_go<__nv_bfloat16>(*p, stream);
}
