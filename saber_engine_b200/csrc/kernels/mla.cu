// Latent attention over a paged cache of latents.
//
// Absorbed form (decoding, short portions, fp32): the query is carried into the latent space, W_uk^T q, so that
// all heads of a row read the same cached row once; the weighted latents are carried out by W_uv.  Rows are
// independent (each knows its sequence and position), so any ragged batch is the same launch; keys may be
// split over CTAs and are merged by the output kernel.
#include "launch.cuh"
#include "mla_device.cuh"

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
  const int m = blockIdx.x;
  if (mla_seq_of_row(p.cu_rows, p.nseq, m) < 0) return;
  const float* x = p.x + static_cast<size_t>(m) * p.ldx;
  const float pos = static_cast<float>(p.pos[m]);
  const int half = p.R / 2, LD = p.CP + p.RP;
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
    for (int i = threadIdx.x; i < p.RP; i += 256) {
      float v = 0.f;
      if (i < p.R) {
        const int f = i < half ? i : i - half;
        float sn, cs;
        sincosf(pos * p.freq[f], &sn, &cs);
        const float a = d[p.C + f], b = d[p.C + f + half];
        v = i < half ? a * cs - b * sn : b * cs + a * sn;
      }
      c[p.CP + i] = from_f<T>(v);
    }
  } else if (slot >= 0 && threadIdx.x == 0 && p.err) {
    atomicCAS(p.err, 0u, static_cast<uint32_t>(kErrBadIndex));
  }
  const int KP = p.expand ? p.DP : p.CP;
  T* q = static_cast<T*>(p.q_eff) + static_cast<size_t>(m) * p.H * (KP + p.RP);
  for (int i = threadIdx.x; i < p.H * p.RP; i += 256) {
    const int h = i / p.RP, k = i - h * p.RP;
    float v = 0.f;
    if (k < p.R) {
      const int f = k < half ? k : k - half;
      float sn, cs;
      sincosf(pos * p.freq[f], &sn, &cs);
      const float* qr = x + p.q_off + h * (p.D + p.R) + p.D;
      const float a = qr[f], b = qr[f + half];
      v = k < half ? a * cs - b * sn : b * cs + a * sn;
    }
    q[static_cast<size_t>(h) * (KP + p.RP) + KP + k] = from_f<T>(v);
  }
  if (p.expand)
    for (int i = threadIdx.x; i < p.H * p.DP; i += 256) {
      const int h = i / p.DP, k = i - h * p.DP;
      q[static_cast<size_t>(h) * (KP + p.RP) + k] = from_f<T>(k < p.D ? x[p.q_off + h * (p.D + p.R) + k] : 0.f);
    }
}

// grid (ceil(CP / 128), H, ceil(M / 8)), 128 threads: q_eff[m][h][r] = sum_d W_uk[h D + d][r] q[m][h][d]
template <typename T>
__global__ void __launch_bounds__(128) mla_absorb_kernel(const __grid_constant__ MlaParams p) {
  pdl_wait();
  extern __shared__ float sm[];                   // [D][8]
  const int h = blockIdx.y, mb = blockIdx.z * 8, rows = min(8, p.M - mb);
  for (int i = threadIdx.x; i < p.D * 8; i += 128) {
    const int d = i >> 3, r = i & 7;
    sm[i] = r < rows ? p.x[static_cast<size_t>(mb + r) * p.ldx + p.q_off + h * (p.D + p.R) + d] : 0.f;
  }
  __syncthreads();
  const int c = blockIdx.x * 128 + threadIdx.x;
  if (c >= p.CP) return;
  float acc[8] = {};
  if (c < p.C) {
    const T* w = static_cast<const T*>(p.w_uk) + static_cast<size_t>(h) * p.D * p.CP + c;
#pragma unroll 4
    for (int d = 0; d < p.D; ++d) {
      const float wv = to_f<T>(w[static_cast<size_t>(d) * p.CP]);
      const float4 a = *reinterpret_cast<const float4*>(sm + d * 8), b = *reinterpret_cast<const float4*>(sm + d * 8 + 4);
      acc[0] = fmaf(wv, a.x, acc[0]); acc[1] = fmaf(wv, a.y, acc[1]); acc[2] = fmaf(wv, a.z, acc[2]); acc[3] = fmaf(wv, a.w, acc[3]);
      acc[4] = fmaf(wv, b.x, acc[4]); acc[5] = fmaf(wv, b.y, acc[5]); acc[6] = fmaf(wv, b.z, acc[6]); acc[7] = fmaf(wv, b.w, acc[7]);
    }
  }
  const int LD = p.CP + p.RP;
#pragma unroll
  for (int r = 0; r < 8; ++r)
    if (r < rows) static_cast<T*>(p.q_eff)[(static_cast<size_t>(mb + r) * p.H + h) * LD + c] = from_f<T>(acc[r]);
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
      rows_s[threadIdx.x] = static_cast<const T*>(p.cache) + (static_cast<size_t>(mla_page_at(p, j, key / p.page)) * p.page + key % p.page) * LD;
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

// grid (ceil(M / 8), H, ceil(V / 64)), 256 threads: merges the key splits of eight rows, carries their latents out
// through W_uv (each weight row is read once for the eight), gates
template <typename T>
__global__ void __launch_bounds__(256) mla_out_kernel(const __grid_constant__ MlaParams p) {
  pdl_wait();
  extern __shared__ float sm[];                   // [8][CP] latents | [8][splits] merge weights
  const int mb = blockIdx.x * 8, h = blockIdx.y, rows = min(8, p.M - mb);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* wt = sm + 8 * p.CP;
  if (warp < rows) {                              // a warp per row: merge weights exp(m_s - max) / sum
    const float* ml = p.ml + (static_cast<size_t>(mb + warp) * p.H + h) * p.splits * 2;
    const bool live = mla_seq_of_row(p.cu_rows, p.nseq, mb + warp) >= 0;
    float mx = -INFINITY, l = 0.f;
    for (int s = lane; s < p.splits; s += 32) mx = fmaxf(mx, live ? ml[s * 2] : -INFINITY);
    mx = mla_warp_max(mx);
    for (int s = lane; s < p.splits; s += 32) l += live && ml[s * 2] > -INFINITY ? ml[s * 2 + 1] * expf(ml[s * 2] - mx) : 0.f;
    l = mla_warp_sum(l);
    for (int s = lane; s < p.splits; s += 32) wt[warp * p.splits + s] = live && ml[s * 2] > -INFINITY ? expf(ml[s * 2] - mx) / l : 0.f;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < 8 * p.CP; i += 256) {
    const int r = i / p.CP, c = i - r * p.CP;
    float v = 0.f;
    if (r < rows) {
      const float* o = p.o_part + (static_cast<size_t>(mb + r) * p.H + h) * p.splits * p.CP + c;
      for (int s = 0; s < p.splits; ++s) {
        const float w = wt[r * p.splits + s];
        if (w != 0.f) v = fmaf(o[static_cast<size_t>(s) * p.CP], w, v);     // (a split without keys, or a padding row, was not written)
      }
    }
    sm[i] = v;
  }
  __syncthreads();
  const int v1 = min(p.V, static_cast<int>(blockIdx.z) * 64 + 64);
  for (int v = blockIdx.z * 64 + warp; v < v1; v += 8) {
    const T* w = static_cast<const T*>(p.w_uv) + (static_cast<size_t>(h) * p.V + v) * p.CP;
    float s[8] = {};
    for (int c = lane; c < p.C; c += 32) {
      const float wv = to_f<T>(w[c]);
#pragma unroll
      for (int r = 0; r < 8; ++r) s[r] = fmaf(wv, sm[r * p.CP + c], s[r]);
    }
#pragma unroll
    for (int r = 0; r < 8; ++r) s[r] = mla_warp_sum(s[r]);
    if (lane < rows) {
      float y = s[0];
#pragma unroll
      for (int r = 1; r < 8; ++r) y = lane == r ? s[r] : y;
      const float g = p.x[static_cast<size_t>(mb + lane) * p.ldx + p.g_off + h * p.V + v];
      operand_store1(p.out, mb + lane, p.out_k0 + h * p.V + v, y / (1.f + expf(-g)));
    }
  }
}

template <typename T>
static int mla_go(const MlaParams& p, cudaStream_t stream) {
  cudaError_t e = launch(mla_prep_kernel<T>, dim3(p.M), dim3(256), 0, stream, 0, p);
  if (e != cudaSuccess) return static_cast<int>(e);
  if (p.expand) return saber_mla_expand_attn(&p, stream);
  e = launch(mla_absorb_kernel<T>, dim3((p.CP + 127) / 128, p.H, (p.M + 7) / 8), dim3(128), p.D * 32, stream, 0, p);
  if (e != cudaSuccess) return static_cast<int>(e);
  if (saber_mla_decode_ok(&p)) {
    const int r = saber_mla_decode_attn(&p, stream);
    if (r != 0) return r;
  } else {
    e = launch(mla_row_attn_kernel<T>, dim3(p.M, p.H, p.splits), dim3(128), (p.CP + p.RP + kRowKeys) * 4, stream, 0, p);
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  return static_cast<int>(launch(mla_out_kernel<T>, dim3((p.M + 7) / 8, p.H, (p.V + 63) / 64), dim3(256), 8 * (p.CP + p.splits) * 4, stream, 0, p));
}

}  // namespace saber

extern "C" int saber_mla_launches(const saber::MlaParams* p) { return p->expand ? 3 : 4; }

extern "C" int saber_mla_launch(const saber::MlaParams* p, cudaStream_t stream) {
  using namespace saber;
  if (p->M <= 0 || p->C > p->CP || p->R > p->RP || (p->R & 1) || p->CP > 128 * kRowMaxC || p->D > 1024 || p->splits < 1 || p->splits > 64 ||
      p->q_eff == nullptr || p->cache == nullptr)
    return static_cast<int>(cudaErrorInvalidValue);
  if (p->expand ? (p->k_exp == nullptr || p->v_exp == nullptr || !saber_mla_expand_ok(p)) : (p->o_part == nullptr || p->ml == nullptr))
    return static_cast<int>(cudaErrorInvalidValue);
  return p->f32 ? mla_go<float>(*p, stream) : mla_go<__nv_bfloat16>(*p, stream);
}
