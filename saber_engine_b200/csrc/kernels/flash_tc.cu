// Causal attention of prompt portions over tiled keys and values, on tcgen05: expanded latents (mla.cu) and
// grouped-query pages (gqa.cu).
//
// A CTA owns 128 query rows of one head and walks the keys its rows can see 128 (two pages) at a time.
//   warp 0     bulk copies: key tiles [k-block of 64][128 keys][128 bytes] and transposed value tiles
//              [page][value row][64 keys], both stored swizzled, two stages each
//   warp 1     one lane issues S = Q K^T into one of two 128-column score buffers, a tile ahead of the softmax,
//              and O += P V with P in tensor memory
//   warps 2-9  softmax, two threads per query row, half of the keys each: scores from tensor memory, running maximum
//              (the halves meet in shared memory), bf16 probabilities back to tensor memory.  O is rescaled only when a row's maximum has grown by more than 2^8 since the
//              factor in use was chosen (the factor cancels in the division at the end).
#include "flash_tc.h"
#include "launch.cuh"
#include "mla_device.cuh"

namespace saber {

constexpr int kTcThreads = 320;
constexpr int kTcKeys = 128;
constexpr float kTcLog2e = 1.4426950408889634f;
constexpr float kTcSlack = 8.f;
constexpr float kTcNone = -1e30f;          // no key seen yet

__device__ __forceinline__ void mma_bf16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t"
      "}\n" ::"r"(d_tmem),
      "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// cap tanh(z s) from 2^(2 z s log2 e): zs is 2 z log2 e.  (Large sums give cap, tiny ones -cap.)
__device__ __forceinline__ float soft_cap(float s, float zs, float cap) { return cap - __fdividef(2.f * cap, 1.f + ex2(s * zs)); }

// tanh(z) = z P(z^2) for |z| <= 0.75 to a relative error of 1e-7: interpolation of tanh(z) / z in the Chebyshev points
// of z^2, in powers of z^2
constexpr float kTanhReach = 0.75f;
constexpr int kTanhTerms = 7;
__constant__ float kTanh[kTanhTerms] = {1.f, -0.33333307505f, 0.13332590461f, -0.05388652161f, 0.02143389918f, -0.00763178663f, 0.00172316108f};

// grid (query tiles of the longest possible portion, H, nseq)
__global__ void __launch_bounds__(kTcThreads) flash_tc_kernel(const __grid_constant__ FlashParams p) {
  pdl_wait();
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t bars[16];
  __shared__ uint32_t tmem_base_s;
  __shared__ volatile uint32_t abort_s[4];          // per pair of softmax warps
  __shared__ float half_s[2][2][128];               // [block parity][half of the keys][row]
  const int h = blockIdx.y, j = blockIdx.z;
  const int r0 = p.cu_rows[j], nrows = p.cu_rows[j + 1] - r0;
  const int tiles = (nrows + 127) / 128;
  if (static_cast<int>(blockIdx.x) >= tiles) return;
  const int qt = tiles - 1 - static_cast<int>(blockIdx.x);          // long rows of keys first
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int DK = p.DK, KB = (DK + 63) >> 6, VP = p.VP;
  const int m0 = r0 + qt * 128, rows = min(128, nrows - qt * 128);
  const int pos0 = p.kv_len[j] - nrows + qt * 128;                  // position of the tile's first row
  const int keys = pos0 + rows;
  const int first = first_key(pos0, p.chunk, p.window);             // first key any row of the tile sees
  const int b0 = first / kTcKeys, blocks = (keys + kTcKeys - 1) / kTcKeys - b0;
  const uint32_t q_s = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t kbytes = static_cast<uint32_t>(KB) * 16384u, vbytes = static_cast<uint32_t>(VP) * 256u;
  const uint32_t k_s = q_s + kbytes, v_s = k_s + 2 * kbytes;
  const uint32_t bar = smem_u32(bars);
  const uint32_t kfull = bar, kfree = bar + 16, vfull = bar + 32, vfree = bar + 48, sfull = bar + 64, sfree = bar + 80, pfull = bar + 96,
                 odone = bar + 104, bend = bar + 112;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(kfull + 8 * i, 1);
      mbar_init(kfree + 8 * i, 1);
      mbar_init(vfull + 8 * i, 1);
      mbar_init(vfree + 8 * i, 1);
      mbar_init(sfull + 8 * i, 1);
      mbar_init(sfree + 8 * i, 8);
    }
    for (int i = 0; i < 4; ++i) abort_s[i] = 0u;
    mbar_init(pfull, 8);
    mbar_init(odone, 1);
    mbar_init(bend, 1);
    mbar_init_fence();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_base_s), 512);
    tmem_relinquish();
  }
  // query tile, swizzled; columns past DK and rows past the live ones are zeros
  const __nv_bfloat16* qg = static_cast<const __nv_bfloat16*>(p.q) + (static_cast<size_t>(m0) * p.H + h) * DK;
  for (int r = warp; r < 128; r += 10)
    for (int c = lane; c < KB * 8; c += 32) {
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < rows && c * 8 < DK) v = *reinterpret_cast<const uint4*>(qg + static_cast<size_t>(r) * p.H * DK + c * 8);
      asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};" ::"r"(q_s + (c >> 3) * 16384 + sw128_offset(r, (c & 7) * 16)), "r"(v.x), "r"(v.y),
                   "r"(v.z), "r"(v.w) : "memory");
    }
  fence_proxy_async_smem();
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tm = tmem_base_s, tm_o = tm + 256, tm_p = tm + 448;

  if (warp == 0) {
    // ---------------------------------------------------------------- copies
    if (lane == 0) {
      const uint8_t* ke = static_cast<const uint8_t*>(p.k);
      const uint8_t* ve = static_cast<const uint8_t*>(p.v);
      const int last = (keys - 1) / 64, g = h / (p.H / p.G);
      int b = 0;
      bool ok = true;
      for (; b < blocks; ++b) {
        const int s = b & 1;
        const uint32_t ph = ((b >> 1) & 1) ^ 1;                     // of the use before this one
        size_t at[2];                                               // (a missing second page: the first again, its keys are masked)
        const int pg = (b0 + b) * 2;
        at[0] = static_cast<size_t>(page_at(p, j, pg)) * p.G + g;
        at[1] = pg + 1 <= last ? static_cast<size_t>(page_at(p, j, pg + 1)) * p.G + g : at[0];
        if (b >= 2 && !mbar_wait(kfree + 8 * s, ph, p.err, kErrWaitEmpty)) { ok = false; break; }
        mbar_arrive_expect_tx(kfull + 8 * s, kbytes);
        for (int kb = 0; kb < KB; ++kb)
          for (int i = 0; i < 2; ++i)
            bulk_g2s(k_s + s * kbytes + kb * 16384 + i * 8192, ke + at[i] * p.k_stride + static_cast<size_t>(kb) * 8192, 8192, kfull + 8 * s);
        if (b >= 2 && !mbar_wait(vfree + 8 * s, ph, p.err, kErrWaitEmpty)) {
          mbar_wait(kfull + 8 * s, (b >> 1) & 1, p.err, kErrWaitDrain);
          ok = false;
          break;
        }
        mbar_arrive_expect_tx(vfull + 8 * s, vbytes);
        for (int i = 0; i < 2; ++i) bulk_g2s(v_s + s * vbytes + i * (vbytes >> 1), ve + at[i] * p.v_stride, vbytes >> 1, vfull + 8 * s);
      }
      if (!ok)                                                      // do not leave while an own copy is in flight
        for (int i = max(0, b - 2); i < b; ++i) {
          mbar_wait(kfull + 8 * (i & 1), (i >> 1) & 1, p.err, kErrWaitDrain);
          mbar_wait(vfull + 8 * (i & 1), (i >> 1) & 1, p.err, kErrWaitDrain);
        }
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      const uint32_t id_s = make_idesc(kCFmtF32, kFmtBF16, kFmtBF16, 128, 128);
      const uint32_t id_o = make_idesc(kCFmtF32, kFmtBF16, kFmtBF16, 128, static_cast<uint32_t>(VP));
      const int steps = DK >> 4;
      auto score = [&](int b) -> bool {                             // S of block b
        const int s = b & 1;
        if (!mbar_wait(kfull + 8 * s, (b >> 1) & 1, p.err, kErrWaitReady)) return false;
        if (b >= 2 && !mbar_wait(sfree + 8 * s, ((b >> 1) & 1) ^ 1, p.err, kErrWaitReady)) return false;
        tc_fence_after_sync();
        for (int t = 0; t < steps; ++t) {
          const uint32_t off = static_cast<uint32_t>(t >> 2) * 16384u + static_cast<uint32_t>(t & 3) * 32u;
          mma_f16_ss(tm + s * 128, make_desc_k128(q_s) + (off >> 4), make_desc_k128(k_s + s * kbytes) + (off >> 4), id_s, t != 0 ? 1u : 0u);
        }
        mma_commit(sfull + 8 * s);
        mma_commit(kfree + 8 * s);
        return true;
      };
      bool ok = score(0);
      for (int b = 0; ok && b < blocks; ++b) {
        if (b + 1 < blocks && !score(b + 1)) { ok = false; break; }
        const int s = b & 1;
        if (!mbar_wait(vfull + 8 * s, (b >> 1) & 1, p.err, kErrWaitReady) || !mbar_wait(pfull, b & 1, p.err, kErrWaitReady)) { ok = false; break; }
        tc_fence_after_sync();
        for (int t = 0; t < 8; ++t) {
          const uint32_t off = static_cast<uint32_t>(t >> 2) * (vbytes >> 1) + static_cast<uint32_t>(t & 3) * 32u;
          mma_bf16_ts(tm_o, tm_p + t * 8, make_desc_k128(v_s + s * vbytes) + (off >> 4), id_o, (b != 0 || t != 0) ? 1u : 0u);
        }
        mma_commit(odone);
        mma_commit(vfree + 8 * s);
      }
      mma_commit(bend);                                             // everything issued has retired before the tensor memory goes back
      mbar_wait(bend, 0, p.err, kErrWaitDrain);
    }
  } else {
    // ---------------------------------------------------------------- softmax
    const int q4 = warp & 3, row = q4 * 32 + lane, half = (warp - 2) >> 2;
    const uint32_t lane_off = static_cast<uint32_t>(q4 * 32) << 16;
    const bool capped = p.softcap > 0.f, series = capped && p.bound > 0.f && fabsf(p.scale) * p.bound <= kTanhReach * p.softcap;
    // scores in the base-2 domain: sc times what v holds (1 where the cap already brought them there)
    const float sc = series ? 1.f : capped ? kTcLog2e : p.scale * kTcLog2e, zs = capped ? 2.f * kTcLog2e * p.scale / p.softcap : 0.f;
    f32x2 co[kTanhTerms];
    {
      const float z2 = capped ? (p.scale / p.softcap) * (p.scale / p.softcap) : 0.f;
      float f = p.scale * kTcLog2e;
#pragma unroll
      for (int i = 0; i < kTanhTerms; ++i) {
        co[i] = pack_f2(kTanh[i] * f, kTanh[i] * f);
        f *= z2;
      }
    }
    // (a row may meet blocks ahead of its first key: the maximum starts finite so that differences stay numbers)
    float mx = kTcNone, used = kTcNone, l = 0.f;
    const int low = first_key(pos0 + row, p.chunk, p.window);       // first key of this row
    const int low_last = first_key(pos0 + q4 * 32 + 31, p.chunk, p.window);
    // A wait that runs out ends both warps of a row: the one that gives up arrives at their next meeting without waiting.
    auto give_up = [&]() {
      abort_s[q4] = 1u;
      __threadfence_block();
      named_bar_arrive(1 + q4, 64);
    };
    bool ok = true;
    for (int b = 0; b < blocks; ++b) {
      const int s = b & 1;
      // (waits are decided by the warp as a whole: tensor-memory accesses need all its lanes together)
      ok = __all_sync(0xffffffffu, mbar_wait(sfull + 8 * s, (b >> 1) & 1, p.err, kErrWaitAcc));
      if (!ok) { give_up(); break; }
      tc_fence_after_sync();
      float v[64];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t r[32];
        tmem_ld32(tm + lane_off + s * 128 + half * 64 + c * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) v[c * 32 + i] = __uint_as_float(r[i]);
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(sfree + 8 * s);
      if (series) {
#pragma unroll
        for (int i = 0; i < 64; i += 2) {
          const f32x2 x = pack_f2(v[i], v[i + 1]), u = mul_f2(x, x);
          f32x2 y = co[kTanhTerms - 1];
#pragma unroll
          for (int t = kTanhTerms - 2; t >= 0; --t) y = fma_f2(y, u, co[t]);
          const float2 f = unpack_f2(mul_f2(x, y));
          v[i] = f.x;
          v[i + 1] = f.y;
        }
      } else if (capped) {
#pragma unroll
        for (int i = 0; i < 64; ++i) v[i] = soft_cap(v[i], zs, p.softcap);
      }
      const int key0 = (b0 + b) * kTcKeys + half * 64;
      const int vis = pos0 + row - key0, low_v = low - key0;        // last and first visible key of this row inside the half block
      if (key0 + 63 > pos0 + q4 * 32) {
#pragma unroll
        for (int i = 0; i < 64; ++i)
          if (i > vis) v[i] = -INFINITY;
      }
      if (low_last > key0) {
#pragma unroll
        for (int i = 0; i < 64; ++i)
          if (i < low_v) v[i] = -INFINITY;
      }
      float m4[4] = {mx, mx, mx, mx};
#pragma unroll
      for (int i = 0; i < 64; ++i) m4[i & 3] = fmaxf(m4[i & 3], v[i]);
      mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
      half_s[s][half][row] = mx;
      named_bar_sync(1 + q4, 64);
      if (abort_s[q4] != 0u) { ok = false; break; }
      mx = fmaxf(mx, half_s[s][half ^ 1][row]);
      // P and O of the block before are consumed
      ok = __all_sync(0xffffffffu, b == 0 || mbar_wait(odone, (b - 1) & 1, p.err, kErrWaitAcc));
      if (!ok) { give_up(); break; }
      const bool grow = b == 0 || (mx - used) * sc > kTcSlack;
      if (__any_sync(0xffffffffu, grow)) {
        const float f = (grow && b > 0) ? ex2((used - mx) * sc) : 1.f;
        if (grow) used = mx;
        l *= b > 0 ? f : 0.f;
        if (b > 0) {
          tc_fence_after_sync();
          for (int c = half * 32; c < VP; c += 64) {                // (the halves take turns over the columns)
            uint32_t r[32];
            tmem_ld32(tm_o + lane_off + c, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * f);
            tmem_st32(tm_o + lane_off + c, r);
          }
          tmem_st_wait();
        }
      }
      const float base = used * sc;
      float sum[4] = {};
      {
        uint32_t r[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const float a = ex2(fmaf(v[2 * i], sc, -base)), e = ex2(fmaf(v[2 * i + 1], sc, -base));
          sum[i & 3] += a + e;
          r[i] = pack2(a, e);
        }
        tmem_st32(tm_p + lane_off + half * 32, r);
      }
      tmem_st_wait();
      l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(pfull);
    }
    if (ok) {
      ok = __all_sync(0xffffffffu, mbar_wait(odone, (blocks - 1) & 1, p.err, kErrWaitAcc));
      if (!ok) give_up();
    }
    if (ok) {
      half_s[blocks & 1][half][row] = l;
      named_bar_sync(1 + q4, 64);
      ok = abort_s[q4] == 0u;
    }
    if (ok) {
      tc_fence_after_sync();
      const int m = m0 + row;
      const bool live = row < rows;
      float den = half_s[blocks & 1][0][row] + half_s[blocks & 1][1][row];
      if (p.sink != nullptr) den += ex2(p.sink[h] * kTcLog2e - used * sc);        // (infinite: the sink takes everything)
      float inv = p.out_scale / den;
      const float* g = p.gate == nullptr ? nullptr : p.gate + static_cast<size_t>(live ? m : m0) * p.ldg + (p.gate_heads ? h : h * p.V);
      if (g != nullptr && p.gate_heads) {
        inv /= 1.f + expf(-g[0]);
        g = nullptr;
      }
      const int k0 = p.out_k0 + h * p.V;
      for (int c = half * 32; c < VP; c += 64) {
        uint32_t r[32];
        __syncwarp();
        tmem_ld32(tm_o + lane_off + c, r);
        tmem_ld_wait();
        if (!live) continue;
        if ((p.V & 7) == 0) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if (c + i * 8 >= p.V) break;
            float y[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] = __uint_as_float(r[i * 8 + e]) * inv;
            if (g != nullptr) {
              const float4 ga = *reinterpret_cast<const float4*>(g + c + i * 8), gb = *reinterpret_cast<const float4*>(g + c + i * 8 + 4);
              const float gg[8] = {ga.x, ga.y, ga.z, ga.w, gb.x, gb.y, gb.z, gb.w};
#pragma unroll
              for (int e = 0; e < 8; ++e) y[e] = y[e] / (1.f + expf(-gg[e]));
            }
            operand_store8(p.out, m, k0 + c + i * 8, y);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c + i < p.V) {
              const float y = __uint_as_float(r[i]) * inv;
              operand_store1(p.out, m, k0 + c + i, g != nullptr ? y / (1.f + expf(-g[c + i])) : y);
            }
        }
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tm, 512);
}

static int flash_tc_smem(int DK, int VP) { return 3 * ((DK + 63) / 64) * 16384 + 2 * VP * 256 + 1024; }

}  // namespace saber

// VP: the accumulator shares tensor memory with two score buffers (256 columns) and the probabilities (64)
bool saber_flash_tc_ok(int page, int DK, int VP, float scale, float softcap) {
  return (scale > 0.f || softcap > 0.f) && page == 64 && (VP & 31) == 0 && VP <= 192 && (DK & 15) == 0 && saber::flash_tc_smem(DK, VP) <= 224 * 1024;
}

int saber_flash_tc(const saber::FlashParams* p, cudaStream_t stream) {
  using namespace saber;
  static bool ready[64];
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return static_cast<int>(cudaErrorInvalidDevice);
  if (!ready[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(flash_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    ready[dev] = true;
  }
  return static_cast<int>(launch(flash_tc_kernel, dim3((p->max_rows + 127) / 128, p->H, p->nseq), dim3(kTcThreads),
                                 flash_tc_smem(p->DK, p->VP), stream, 0, *p));
}
