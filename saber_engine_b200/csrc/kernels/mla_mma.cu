// Latent attention on the tensor cores (bf16 operands, fp32 scores, softmax and accumulators).
//
// decode  absorbed form.  The heads of a row are the rows of the query tile and every key row is read once
//         for all of them: scores against [latent | rotated part], values are the latent columns of the same
//         shared-memory tile.  64 keys at a time, double buffered; keys are split over CTAs.
// expand  keys and values of the pages a step sees, [W_uk c | rotated part] and W_uv c, into scratch pages.
// flash   causal attention of prompt portions over the scratch pages: 128 query rows of one head per CTA,
//         16 per warp, one page of 64 keys at a time, running softmax in the base-2 domain.
#include "flash_tc.h"
#include "launch.cuh"
#include "mla_device.cuh"

namespace saber {

constexpr int kKeys = 64;
constexpr float kLog2e = 1.4426950408889634f;

// ------------------------------------------------------------------------------------ decode
// grid (M, head groups, splits), 256 threads.  MT: 16-head tiles of the group.  NC: 8-column groups of the
// latent per warp (CP <= 64 NC).
template <int MT, int NC>
__global__ void __launch_bounds__(256) mla_decode_kernel(const __grid_constant__ MlaParams p) {
  pdl_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  const int m = blockIdx.x, h0 = blockIdx.y * MT * 16, sp = blockIdx.z;
  const int j = mla_seq_of_row(p.cu_rows, p.nseq, m);
  if (j < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int LD = p.CP + p.RP;
  const uint32_t rs = static_cast<uint32_t>(LD) * 2u + 16u;         // row stride: an odd number of 16-byte units
  const int nh = min(MT * 16, p.H - h0);
  const uint32_t q_s = smem_u32(smem);
  const uint32_t k_s = q_s + MT * 16 * rs;                          // two tiles of 64 rows
  const uint32_t p_s = k_s + 2 * kKeys * rs;                        // probabilities, bf16 [MT * 16][64 + 8]
  float* s_f = reinterpret_cast<float*>(smem + (MT * 16 + 2 * kKeys) * rs + MT * 16 * 144);   // partial scores [2][MT * 16][64 + 4]
  float* corr_s = s_f + 2 * MT * 16 * 68;                           // [MT * 16]
  const int keys = p.pos[m] + 1;
  const int per = ((keys + p.splits - 1) / p.splits + kKeys - 1) / kKeys * kKeys;
  const int k0 = sp * per, k1 = min(keys, k0 + per);
  const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(p.cache);
  const int chunks = LD / 8;

  const __nv_bfloat16* qg = static_cast<const __nv_bfloat16*>(p.q_eff) + (static_cast<size_t>(m) * p.H + h0) * LD;
  for (int i = threadIdx.x; i < MT * 16 * chunks; i += 256) {
    const int r = i / chunks, c = i - r * chunks;
    cp16(q_s + r * rs + c * 16, qg + static_cast<size_t>(min(r, nh - 1)) * LD + c * 8, r < nh);
  }
  auto fetch = [&](int kb, int buf) {
    const uint32_t dst = k_s + buf * kKeys * rs;
    for (int r = warp; r < kKeys; r += 8) {                         // a warp per key row
      const int key = kb + r;
      const bool live = key < k1;
      const int at = live ? key : k0;
      const __nv_bfloat16* src = cache + (static_cast<size_t>(page_at(p, j, at / p.page)) * p.page + at % p.page) * LD;
      for (int c = lane; c < chunks; c += 32) cp16(dst + r * rs + c * 16, src + c * 8, live);
    }
    cp_commit();
  };
  float o[MT][NC][4] = {};
  float mx[2 * MT], l[2 * MT];                                      // rows warp, warp + 8, ... of the tile
#pragma unroll
  for (int i = 0; i < 2 * MT; ++i) { mx[i] = -INFINITY; l[i] = 0.f; }
  if (k0 < k1) {
    fetch(k0, 0);
  } else {
    cp_commit();
    cp_wait<0>();
  }
  int buf = 0;
  for (int kb = k0; kb < k1; kb += kKeys, buf ^= 1) {
    if (kb + kKeys < k1) {
      fetch(kb + kKeys, buf ^ 1);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const uint32_t kt = k_s + buf * kKeys * rs;
    // scores of 16 keys (warp & 3) over one half of the score dimension (warp >> 2) for every head tile
    {
      float s[MT][2][4] = {};
      const int steps = LD / 16, half0 = (steps + 1) / 2;
      const int s0 = warp < 4 ? 0 : half0, s1 = warp < 4 ? half0 : steps;
      const int kg = (warp & 3) * 16;
      const uint32_t a_row = q_s + (lane & 15) * rs + ((lane >> 4) << 4);
      const uint32_t b_row = kt + (kg + ((lane >> 4) << 3) + (lane & 7)) * rs + (((lane >> 3) & 1) << 4);
#pragma unroll 4
      for (int st = s0; st < s1; ++st) {
        uint32_t b[4];
        ldsm4(b, b_row + st * 32);
#pragma unroll
        for (int t = 0; t < MT; ++t) {
          uint32_t a[4];
          ldsm4(a, a_row + t * 16 * rs + st * 32);
          mma16816(s[t][0], a, b[0], b[1]);
          mma16816(s[t][1], a, b[2], b[3]);
        }
      }
      float* dst = s_f + (warp >> 2) * MT * 16 * 68;
      const int r = lane >> 2;
#pragma unroll
      for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int c = kg + i * 8 + (lane & 3) * 2;
          *reinterpret_cast<float2*>(dst + (t * 16 + r) * 68 + c) = make_float2(s[t][i][0], s[t][i][1]);
          *reinterpret_cast<float2*>(dst + (t * 16 + r + 8) * 68 + c) = make_float2(s[t][i][2], s[t][i][3]);
        }
    }
    __syncthreads();
    // running softmax: warp w owns rows w, w + 8, ...
    const int n = min(kKeys, k1 - kb);
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i) {
      const int r = warp + 8 * i;
      float2 v = *reinterpret_cast<const float2*>(s_f + r * 68 + lane * 2);
      const float2 v2 = *reinterpret_cast<const float2*>(s_f + (MT * 16 + r) * 68 + lane * 2);
      v.x += v2.x;
      v.y += v2.y;
      const float a = lane * 2 < n ? v.x * p.scale : -INFINITY, b = lane * 2 + 1 < n ? v.y * p.scale : -INFINITY;
      const float mn = fmaxf(mx[i], mla_warp_max(fmaxf(a, b)));
      const float ea = ex2((a - mn) * kLog2e), eb = ex2((b - mn) * kLog2e);
      const float corr = ex2((mx[i] - mn) * kLog2e);
      l[i] = l[i] * corr + mla_warp_sum(ea + eb);
      mx[i] = mn;
      asm volatile("st.shared.b32 [%0], %1;" ::"r"(p_s + r * 144 + lane * 4), "r"(pack2(ea, eb)) : "memory");
      if (lane == 0) corr_s[r] = corr;
    }
    __syncthreads();
    // values: this warp's latent columns
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      const float c0 = corr_s[t * 16 + (lane >> 2)], c1 = corr_s[t * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int i = 0; i < NC; ++i) { o[t][i][0] *= c0; o[t][i][1] *= c0; o[t][i][2] *= c1; o[t][i][3] *= c1; }
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t a[MT][4];
#pragma unroll
      for (int t = 0; t < MT; ++t) ldsm4(a[t], p_s + (t * 16 + (lane & 15)) * 144 + ks * 32 + ((lane >> 4) << 4));
#pragma unroll
      for (int i = 0; i < NC; i += 2) {
        const int col = (warp * NC + i) * 8;
        if (col < p.CP) {                                           // CP is a multiple of 16: column pairs are whole
          uint32_t b[4];
          ldsm4_t(b, kt + (ks * 16 + (lane & 15)) * rs + col * 2 + ((lane >> 4) << 4));
#pragma unroll
          for (int t = 0; t < MT; ++t) {
            mma16816(o[t][i], a[t], b[0], b[1]);
            mma16816(o[t][i + 1], a[t], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int t = 0; t < MT; ++t)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int h = t * 16 + (lane >> 2) + half * 8;
      if (h < nh) {
        float* d = p.o_part + ((static_cast<size_t>(m) * p.H + h0 + h) * p.splits + sp) * p.CP;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
          const int col = (warp * NC + i) * 8 + (lane & 3) * 2;
          if (col < p.CP) *reinterpret_cast<float2*>(d + col) = make_float2(o[t][i][half * 2], o[t][i][half * 2 + 1]);
        }
      }
    }
#pragma unroll
  for (int i = 0; i < 2 * MT; ++i) {
    const int h = warp + 8 * i;
    if (lane == 0 && h < nh) {
      float* d = p.ml + ((static_cast<size_t>(m) * p.H + h0 + h) * p.splits + sp) * 2;
      d[0] = mx[i];
      d[1] = l[i];
    }
  }
}

static int decode_smem(const MlaParams& p, int mt) {
  const int rs = (p.CP + p.RP) * 2 + 16;
  return (mt * 16 + 2 * kKeys) * rs + mt * 16 * (144 + 2 * 68 * 4 + 4);
}
static int decode_tiles(const MlaParams& p) {
  const int mt = p.H <= 16 ? 1 : (p.H <= 32 || p.H > 48 ? 2 : 3);
  return mt == 3 && decode_smem(p, 3) > 226 * 1024 ? 2 : mt;
}
template <int MT, int NC>
static int decode_go(const MlaParams& p, cudaStream_t stream) {
  static bool ready[64];
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return static_cast<int>(cudaErrorInvalidDevice);
  if (!ready[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(mla_decode_kernel<MT, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    ready[dev] = true;
  }
  return static_cast<int>(launch(mla_decode_kernel<MT, NC>, dim3(p.M, (p.H + MT * 16 - 1) / (MT * 16), p.splits), dim3(256),
                                 decode_smem(p, MT), stream, 0, p));
}
template <int NC>
static int decode_mt(const MlaParams& p, int mt, cudaStream_t s) {
  return mt == 1 ? decode_go<1, NC>(p, s) : mt == 2 ? decode_go<2, NC>(p, s) : decode_go<3, NC>(p, s);
}

// ------------------------------------------------------------------------------------ expand
// Work items, dealt round-robin to a resident grid: (two pages of a sequence) x (128 weight rows of W_uk, then of
// W_uv, then one item that copies the rotated part and clears padding columns).
// Element of a key row in the tiles of the tcgen05 kernel: [page][head][k-block of 64][64 keys][128 bytes], 16-byte chunks
// XOR (key & 7).
__device__ __forceinline__ size_t k_tile_at(const MlaParams& p, int pg, int h, int key, int d) {
  const int KB = (p.DP + p.RP + 63) >> 6;
  return ((static_cast<size_t>(pg) * p.H + h) * KB + (d >> 6)) * 4096 + key * 64 + (((((d & 63) >> 3) ^ key) & 7) << 3) + (d & 7);
}
constexpr int kExpStride = 144;                    // 64 bf16 + 16 bytes
constexpr int kExpStage = 2 * 128 * kExpStride;    // latents, weights

__global__ void __launch_bounds__(256) mla_expand_kernel(const __grid_constant__ MlaParams p) {
  pdl_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  const uint32_t base = smem_u32(smem);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int wm = warp & 3, wn = warp >> 2;
  const int LD = p.CP + p.RP, DK = p.DP + p.RP;
  const int nk = (p.H * p.D + 127) / 128, nv = (p.H * p.V + 127) / 128, per = nk + nv + 1;
  const int kc = (p.CP + 63) / 64;
  const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(p.cache);
  __nv_bfloat16* ke = static_cast<__nv_bfloat16*>(p.k_exp);
  __nv_bfloat16* ve = static_cast<__nv_bfloat16*>(p.v_exp);
  int pairs = 0;
  for (int j = 0; j < p.nseq; ++j)
    if (p.cu_rows[j + 1] > p.cu_rows[j]) pairs += (p.kv_len[j] + 127) / 128;
  for (int item = blockIdx.x; item < pairs * per; item += gridDim.x) {
    const int tile = item / pairs;                 // pages run fastest: a weight tile is reused from L2
    int pr = item - tile * pairs, j = 0;
    for (;; ++j) {
      const int n = p.cu_rows[j + 1] > p.cu_rows[j] ? (p.kv_len[j] + 127) / 128 : 0;
      if (pr < n) break;
      pr -= n;
    }
    const int len = p.kv_len[j];
    int page[2];
    page[0] = page_at(p, j, pr * 2);
    page[1] = pr * 128 + 64 < len ? page_at(p, j, pr * 2 + 1) : -1;
    if (tile == per - 1) {
      const int rot8 = p.RP / 8;
      for (int i = threadIdx.x; i < 128 * p.H; i += 256) {
        const int r = i / p.H, h = i - r * p.H, pg = page[r >> 6];
        if (pg < 0) continue;
        const __nv_bfloat16* src = cache + (static_cast<size_t>(pg) * 64 + (r & 63)) * LD + p.CP;
        if (p.expand == 2) {
          for (int c = 0; c < rot8; ++c)
            *reinterpret_cast<uint4*>(ke + k_tile_at(p, pg, h, r & 63, p.DP + c * 8)) = reinterpret_cast<const uint4*>(src)[c];
          continue;
        }
        __nv_bfloat16* d = ke + ((static_cast<size_t>(pg) * p.H + h) * 64 + (r & 63)) * DK;
        for (int c = 0; c < rot8; ++c) reinterpret_cast<uint4*>(d + p.DP)[c] = reinterpret_cast<const uint4*>(src)[c];
        for (int c = p.D; c < p.DP; ++c) d[c] = __float2bfloat16(0.f);
        __nv_bfloat16* v = ve + ((static_cast<size_t>(pg) * p.H + h) * 64 + (r & 63)) * p.VP;
        for (int c = p.V; c < p.VP; ++c) v[c] = __float2bfloat16(0.f);
      }
      continue;
    }
    const bool isk = tile < nk;
    const int n0 = (isk ? tile : tile - nk) * 128, N = p.H * (isk ? p.D : p.V), per_h = isk ? p.D : p.V;
    const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(isk ? p.w_uk : p.w_uv);
    const bool vt = !isk && p.expand == 2;         // values transposed: weight rows are the rows of the product
    auto fetch = [&](int c, int buf) {
      const uint32_t dst = base + buf * kExpStage;
      for (int i = threadIdx.x; i < 2048; i += 256) {
        const int r = (i & 1023) >> 3, ch = i & 7, col = c * 64 + ch * 8;
        const bool ina = i < 1024;
        const int pg = page[r >> 6];
        const bool live = col < p.CP && (ina ? pg >= 0 : n0 + r < N);
        const __nv_bfloat16* src = !live ? w : ina ? cache + (static_cast<size_t>(pg) * 64 + (r & 63)) * LD + col
                                                   : w + static_cast<size_t>(n0 + r) * p.CP + col;
        cp16(dst + (ina ? 0 : 128 * kExpStride) + r * kExpStride + ch * 16, src, live);
      }
      cp_commit();
    };
    float acc[2][8][4] = {};
    fetch(0, 0);
    if (kc > 1) fetch(1, 1);
    for (int c = 0; c < kc; ++c) {
      if (c + 2 < kc) fetch(c + 2, (c + 2) % 3);
      if (c + 2 < kc) cp_wait<2>(); else if (c + 1 < kc) cp_wait<1>(); else cp_wait<0>();
      __syncthreads();
      const uint32_t lat_s = base + (c % 3) * kExpStage, wgt_s = lat_s + 128 * kExpStride;
      const uint32_t a_s = vt ? wgt_s : lat_s, b_s = vt ? lat_s : wgt_s;
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        uint32_t a[2][4];
#pragma unroll
        for (int t = 0; t < 2; ++t) ldsm4(a[t], a_s + (wm * 32 + t * 16 + (lane & 15)) * kExpStride + ks * 32 + ((lane >> 4) << 4));
#pragma unroll
        for (int i = 0; i < 8; i += 2) {
          uint32_t b[4];
          ldsm4(b, b_s + (wn * 64 + i * 8 + ((lane >> 4) << 3) + (lane & 7)) * kExpStride + ks * 32 + (((lane >> 3) & 1) << 4));
#pragma unroll
          for (int t = 0; t < 2; ++t) {
            mma16816(acc[t][i], a[t], b[0], b[1]);
            mma16816(acc[t][i + 1], a[t], b[2], b[3]);
          }
        }
      }
      __syncthreads();
    }
    if (p.expand == 2) {
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = wm * 32 + t * 16 + (lane >> 2) + half * 8;
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const int q = wn * 64 + i * 8 + (lane & 3) * 2;
            const int n = n0 + (vt ? r : q), key = vt ? q : r, pg = page[key >> 6];
            if (pg < 0 || n >= N) continue;
            const int h = n / per_h, d = n - h * per_h;
            const float x = acc[t][i][half * 2], y = acc[t][i][half * 2 + 1];
            if (vt) {
              __nv_bfloat16* o = ve + ((static_cast<size_t>(pg) * p.H + h) * p.VP + d) * 64 + (((((key & 63) >> 3) ^ d) & 7) << 3) + (key & 7);
              *reinterpret_cast<uint32_t*>(o) = pack2(x, y);
            } else if ((per_h & 1) == 0) {
              *reinterpret_cast<uint32_t*>(ke + k_tile_at(p, pg, h, key & 63, d)) = pack2(x, y);
            } else {
              ke[k_tile_at(p, pg, h, key & 63, d)] = __float2bfloat16(x);
              if (n + 1 < N) {
                const int h1 = (n + 1) / per_h;
                ke[k_tile_at(p, pg, h1, key & 63, n + 1 - h1 * per_h)] = __float2bfloat16(y);
              }
            }
          }
        }
      continue;
    }
    const bool even = (per_h & 1) == 0;
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = wm * 32 + t * 16 + (lane >> 2) + half * 8, pg = page[r >> 6];
        if (pg < 0) continue;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int n = n0 + wn * 64 + i * 8 + (lane & 3) * 2;
          if (n >= N) continue;
          const int h = n / per_h, d = n - h * per_h;
          const int width = isk ? DK : p.VP;
          __nv_bfloat16* o = (isk ? ke : ve) + ((static_cast<size_t>(pg) * p.H + h) * 64 + (r & 63)) * width + d;
          const float x = acc[t][i][half * 2], y = acc[t][i][half * 2 + 1];
          if (even) {
            *reinterpret_cast<uint32_t*>(o) = pack2(x, y);
          } else {
            o[0] = __float2bfloat16(x);
            if (n + 1 < N) {
              const int h1 = (n + 1) / per_h, d1 = n + 1 - h1 * per_h;
              ((isk ? ke : ve) + ((static_cast<size_t>(pg) * p.H + h1) * 64 + (r & 63)) * width)[d1] = __float2bfloat16(y);
            }
          }
        }
      }
  }
}

// ------------------------------------------------------------------------------------ flash
// grid (query tiles of the longest possible portion, H, nseq), 256 threads.  NV: 8-column groups of a value.
constexpr int kQRows = 128;

template <int NV>
__global__ void __launch_bounds__(256) mla_flash_kernel(const __grid_constant__ MlaParams p) {
  pdl_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  const int h = blockIdx.y, j = blockIdx.z;
  const int r0 = p.cu_rows[j], nrows = p.cu_rows[j + 1] - r0;
  const int tiles = (nrows + kQRows - 1) / kQRows;
  if (static_cast<int>(blockIdx.x) >= tiles) return;
  const int qt = tiles - 1 - static_cast<int>(blockIdx.x);          // long rows of keys first
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int DK = p.DP + p.RP, kch = DK / 8;
  constexpr int VP = NV * 8, vch = NV;
  const uint32_t ks_ = static_cast<uint32_t>(DK) * 2u + 16u;
  constexpr uint32_t vs_ = VP * 2u + 16u;
  const uint32_t q_s = smem_u32(smem);
  const uint32_t kv_s = q_s + kQRows * ks_;
  const uint32_t stage = kKeys * (ks_ + vs_);
  const __nv_bfloat16* ke = static_cast<const __nv_bfloat16*>(p.k_exp);
  const __nv_bfloat16* ve = static_cast<const __nv_bfloat16*>(p.v_exp);
  const int m0 = r0 + qt * kQRows, rows = min(kQRows, nrows - qt * kQRows);
  const int pos0 = p.kv_len[j] - nrows + qt * kQRows;               // position of the tile's first row
  const int keys = pos0 + rows;
  const int blocks = (keys + kKeys - 1) / kKeys;

  const __nv_bfloat16* qg = static_cast<const __nv_bfloat16*>(p.q_eff) + (static_cast<size_t>(m0) * p.H + h) * DK;
  for (int i = threadIdx.x; i < kQRows * kch; i += 256) {
    const int r = i / kch, c = i - r * kch;
    cp16(q_s + r * ks_ + c * 16, qg + static_cast<size_t>(min(r, rows - 1)) * p.H * DK + c * 8, r < rows);
  }
  int next_page = page_at(p, j, 0);                             // looked up one block ahead of its copies
  auto fetch = [&](int b) {
    const size_t pg = static_cast<size_t>(next_page) * p.H + h;
    if (b + 1 < blocks) next_page = page_at(p, j, b + 1);
    const __nv_bfloat16* kg = ke + pg * kKeys * DK;
    const __nv_bfloat16* vg = ve + pg * kKeys * VP;
    const uint32_t kd = kv_s + (b & 1) * stage, vd = kd + kKeys * ks_;
#pragma unroll 4
    for (int r = warp; r < kKeys; r += 8)                           // a warp per key row
      for (int c = lane; c < kch; c += 32) cp16(kd + r * ks_ + c * 16, kg + r * DK + c * 8, true);
    constexpr int kPer = vch < 32 ? 32 / vch : 1;                   // value rows a warp copies at a time
#pragma unroll
    for (int r0v = 0; r0v < kKeys; r0v += 8 * kPer) {
      const int r = r0v + warp * kPer + lane / (vch < 32 ? vch : 32);
      const bool live = b * kKeys + r < keys;                       // rows never written must not reach a product (0 x NaN)
      for (int c = lane % (vch < 32 ? vch : 32); c < vch; c += 32) cp16(vd + r * vs_ + c * 16, vg + r * VP + c * 8, live);
    }
    cp_commit();
  };
  float o[NV][4] = {};
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const float sc = p.scale * kLog2e;
  const int row = warp * 16 + (lane >> 2);                          // and row + 8
  fetch(0);
  for (int b = 0; b < blocks; ++b) {
    if (b + 1 < blocks) {
      fetch(b + 1);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const uint32_t kd = kv_s + (b & 1) * stage, vd = kd + kKeys * ks_;
    float s[8][4] = {};
    const uint32_t a_row = q_s + (warp * 16 + (lane & 15)) * ks_ + ((lane >> 4) << 4);
    const uint32_t b_row = kd + (((lane >> 4) << 3) + (lane & 7)) * ks_ + (((lane >> 3) & 1) << 4);
    // fragments of the next step are requested before the products of this one
    uint32_t fa[4], fb[4][4];
    ldsm4(fa, a_row);
#pragma unroll
    for (int i = 0; i < 4; ++i) ldsm4(fb[i], b_row + i * 16 * ks_);
#pragma unroll 4
    for (int kk = 16; kk <= DK; kk += 16) {
      uint32_t ca[4], cb[4][4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        ca[x] = fa[x];
#pragma unroll
        for (int i = 0; i < 4; ++i) cb[i][x] = fb[i][x];
      }
      // (past the last step: the first fragments again, unused)
      ldsm4(fa, a_row + (kk < DK ? kk : 0) * 2);
#pragma unroll
      for (int i = 0; i < 4; ++i) ldsm4(fb[i], b_row + i * 16 * ks_ + (kk < DK ? kk : 0) * 2);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        mma16816(s[2 * i], ca, cb[i][0], cb[i][1]);
        mma16816(s[2 * i + 1], ca, cb[i][2], cb[i][3]);
      }
    }
    const int kb = b * kKeys;
    const bool edge = kb + kKeys - 1 > pos0 + warp * 16;            // some key lies past some row of this warp
    if (edge) {
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (kb + i * 8 + (lane & 3) * 2 + (e & 1) > pos0 + row + (e >> 1) * 8) s[i][e] = -INFINITY;
    }
    // running maximum in unscaled scores: needs scale > 0 (checked on the host)
    float mn[2] = {mx[0], mx[1]};
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) mn[e >> 1] = fmaxf(mn[e >> 1], s[i][e]);
    float corr[2], base[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mn[r] = fmaxf(mn[r], __shfl_xor_sync(0xffffffffu, mn[r], 1));
      mn[r] = fmaxf(mn[r], __shfl_xor_sync(0xffffffffu, mn[r], 2));
      corr[r] = ex2((mx[r] - mn[r]) * sc);                          // (key 0 is visible to every row: mn is finite)
      base[r] = mn[r] * sc;
      mx[r] = mn[r];
    }
    float sum[2] = {0.f, 0.f};
    uint32_t pa[4][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      float e4[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        e4[e] = ex2(fmaf(s[i][e], sc, -base[e >> 1]));
        sum[e >> 1] += e4[e];
      }
      pa[i >> 1][(i & 1) * 2] = pack2(e4[0], e4[1]);
      pa[i >> 1][(i & 1) * 2 + 1] = pack2(e4[2], e4[3]);
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) l[r] = l[r] * corr[r] + sum[r];
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int i = 0; i < NV; ++i) { o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
    }
    const uint32_t v_row = vd + (lane & 15) * vs_ + ((lane >> 4) << 4);
#pragma unroll
    for (int ks = 0; ks < 4; ++ks)
#pragma unroll
      for (int i = 0; i < NV; i += 2) {
        uint32_t bb[4];
        ldsm4_t(bb, v_row + ks * 16 * vs_ + i * 16);
        mma16816(o[i], pa[ks], bb[0], bb[1]);
        mma16816(o[i + 1], pa[ks], bb[2], bb[3]);
      }
    __syncthreads();
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int rr = row + r * 8;
    if (rr >= rows) continue;
    const float inv = 1.f / l[r];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int v = i * 8 + (lane & 3) * 2;
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (v + e < p.V) operand_store1(p.out, m0 + rr, p.out_k0 + h * p.V + v + e, o[i][r * 2 + e] * inv / (1.f + expf(-mla_gate(p, m0 + rr, h, v + e))));
    }
  }
}

static int flash_smem(const MlaParams& p) {
  const int ks = (p.DP + p.RP) * 2 + 16, vs = p.VP * 2 + 16;
  return kQRows * ks + 2 * kKeys * (ks + vs);
}
template <int NV>
static int flash_go(const MlaParams& p, cudaStream_t stream) {
  static bool ready[64];
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return static_cast<int>(cudaErrorInvalidDevice);
  if (!ready[dev]) {
    cudaError_t e = cudaFuncSetAttribute(mla_flash_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(mla_expand_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 3 * kExpStage);
    if (e != cudaSuccess) return static_cast<int>(e);
    ready[dev] = true;
  }
  cudaError_t e = launch(mla_expand_kernel, dim3(2 * 148), dim3(256), 3 * kExpStage, stream, 0, p);
  if (e == cudaSuccess && p.expand == 2) {
    FlashParams f = {};
    f.out_scale = 1.f;
    f.q = p.q_eff;
    f.k = p.k_exp;
    f.v = p.v_exp;
    f.k_stride = static_cast<size_t>((p.DP + p.RP + 63) / 64) * 8192;
    f.v_stride = static_cast<size_t>(p.VP) * 128;
    f.gate = p.x + p.g_off;
    f.ldg = p.ldx;
    f.gate_heads = p.gate_heads;
    f.cu_rows = p.cu_rows;
    f.kv_len = p.kv_len;
    f.block_table = p.block_table;
    f.out = p.out;
    f.out_k0 = p.out_k0;
    f.nseq = p.nseq;
    f.H = f.G = p.H;
    f.DK = p.DP + p.RP;
    f.V = p.V;
    f.VP = p.VP;
    f.n_blocks = p.n_blocks;
    f.max_blocks = p.max_blocks;
    f.max_rows = p.max_rows;
    f.scale = p.scale;
    f.err = p.err;
    return saber_flash_tc(&f, stream);
  }
  if (e == cudaSuccess)
    e = launch(mla_flash_kernel<NV>, dim3((p.max_rows + kQRows - 1) / kQRows, p.H, p.nseq), dim3(256), flash_smem(p), stream, 0, p);
  return static_cast<int>(e);
}

}  // namespace saber

bool saber_mla_decode_ok(const saber::MlaParams* p) {
  return !p->f32 && p->CP <= 512 && (p->CP & 15) == 0 && (p->RP & 15) == 0 &&
         saber::decode_smem(*p, saber::decode_tiles(*p)) <= 226 * 1024;
}

int saber_mla_decode_attn(const saber::MlaParams* p, cudaStream_t s) {
  const int mt = saber::decode_tiles(*p);
  return p->CP <= 128 ? saber::decode_mt<2>(*p, mt, s) : p->CP <= 256 ? saber::decode_mt<4>(*p, mt, s) : saber::decode_mt<8>(*p, mt, s);
}

// Value sizes and shared-memory needs the expanded form takes on: 2 on tcgen05, 1 on mma.sync, 0 not at all (the
// absorbed form has no such limit).
extern "C" int saber_mla_expand_ok(const saber::MlaParams* p) {
  const bool vp = p->VP == 32 || p->VP == 64 || p->VP == 128 || p->VP == 256;
  if (!p->f32 && p->VP <= 128 && saber_flash_tc_ok(p->page, p->DP + p->RP, p->VP, p->scale, 0.f) && ((p->DP | p->RP | p->CP) & 15) == 0) return 2;
  return !p->f32 && p->scale > 0.f && vp && p->page == saber::kKeys && ((p->DP | p->RP | p->CP) & 15) == 0 && saber::flash_smem(*p) <= 226 * 1024;
}

int saber_mla_expand_attn(const saber::MlaParams* p, cudaStream_t s) {
  switch (p->VP) {
    case 32: return saber::flash_go<4>(*p, s);
    case 64: return saber::flash_go<8>(*p, s);
    case 128: return saber::flash_go<16>(*p, s);
    case 256: return saber::flash_go<32>(*p, s);
    default: return static_cast<int>(cudaErrorInvalidValue);
  }
}
