// Decayed outer products over prompt portions on the tensor cores: 64 tokens at a time, the state in registers.
//
// With q, k, v in bf16 and everything else in fp32, token i of a chunk reads
//     o_i = sum_{j<=i} D_ij w_j (q_i . k_j) v_j  +  A_i S_0^T q_i  +  skip v_i
// and the chunk leaves  S = A_64 S_0 + sum_j B_j w_j k_j v_j^T.  D_ij, A_i and B_j are the decays between two tokens,
// from the start of the chunk and to its end: exponentials of sums of the logarithms of the tokens in between, added up
// as such (inside sixteen tokens, over whole sixteens), never as a difference of prefix sums, so that a token that
// forgets everything costs its neighbours no digits.
//
// fp32 factors meet bf16 ones in `mma.sync`: they are written as a sum of three bf16 values (24 bits, the fp32
// mantissa), three products with fp32 accumulation.  Those are the pair weights P_ij, the state, and B_j w_j v_j.
//
//   prep   convolution, silu -> q, k, v tiles in the order the scan's fragments want them; the tables of decays
//   scan   a CTA per (sequence, head, 64 value columns); a pair of warps holds 16 columns of the state, half of the keys
//          each, as accumulator fragments that are the operand fragments of the next read-out (the halves of a read-out
//          meet in shared memory).  Tiles of the next chunk arrive by bulk copies meanwhile.
#include "launch.cuh"
#include "mla_device.cuh"
#include "ssd_chunk.h"
#include "ssd_device.cuh"

namespace saber {

constexpr int kTok = 64;                 // tokens of a chunk
constexpr int kSlice = 64;               // value columns of a scan CTA
constexpr int kRun = 16;                 // rows a thread of the prep kernel walks

// Chunks of sequence j occupy the slots from (first row / 64) + j on.
__device__ __forceinline__ int chunk_slot(int r0, int j) { return r0 / kTok + j; }
// element of a tile of 64 rows: [64-column block][row][128 bytes], 16-byte pieces XOR (row & 7)
__device__ __forceinline__ int tile_at(int row, int c) { return ((c >> 6) * kTok + row) * 64 + (((((c & 63) >> 3) ^ row) & 7) << 3) + (c & 7); }

// Decays of a chunk, weights included (a bulk copy).
struct ChunkTables {
  float diag[4][16][20];                 // [sixteen][i][j] D_ij w_j of two tokens of the same sixteen, 0 above the diagonal
  float row[kTok];                       // from the start of a token's sixteen to it
  float start[kTok];                     // A_i
  float col[3][kTok];                    // from token j of an earlier sixteen to the start of sixteen a + 1, times w_j
  float end[kTok];                       // B_j w_j
};
static_assert(sizeof(ChunkTables) % 16 == 0, "");

struct ChunkLayout {                     // of a slot, in bytes
  size_t v, gates, bytes;
};
__host__ __device__ inline ChunkLayout chunk_layout(const SsdParams& p) {
  const size_t vs = static_cast<size_t>((p.VP + kSlice - 1) / kSlice);
  ChunkLayout l;
  l.v = static_cast<size_t>(p.HK) * 2 * p.DP * kTok * 2;            // [HK][q | k][DP / 64] tiles
  l.gates = l.v + static_cast<size_t>(p.H) * vs * kTok * kSlice * 2;    // [H][slices] tiles
  l.bytes = l.gates + static_cast<size_t>(p.H) * sizeof(ChunkTables);   // [H]
  return l;
}

// grid (slots, channel groups + head groups, 4), 128 threads: a thread per (padded channel, 16 rows); then per (head, row)
template <int TAPS>
__global__ void __launch_bounds__(128) ssd_chunk_prep_kernel(const __grid_constant__ SsdParams p) {
  pdl_wait();
  int j = 0, c = 0;
  bool found = false;
  for (; j < p.nseq; ++j) {
    const int r0 = p.cu_rows[j], n = p.cu_rows[j + 1] - r0;
    c = static_cast<int>(blockIdx.x) - chunk_slot(r0, j);
    if (c >= 0 && c * kTok < n) { found = true; break; }
  }
  if (!found) return;
  const int slot = ssd_slot(p, j);
  if (slot < 0) return;
  const int t0 = c * kTok, m0 = p.cu_rows[j] + t0, live = min(kTok, p.cu_rows[j + 1] - m0);
  const ChunkLayout lay = chunk_layout(p);
  uint8_t* base = reinterpret_cast<uint8_t*>(p.chunk) + blockIdx.x * lay.bytes;
  const int vs = (p.VP + kSlice - 1) / kSlice, nk = p.HK * p.DP, total = 2 * nk + p.H * vs * kSlice;
  const int groups = (total + 127) / 128;
  if (static_cast<int>(blockIdx.y) >= groups) {
    __shared__ float la_s[2][kTok], total_s[2][4];
    const int hh = threadIdx.x / kTok, h = (blockIdx.y - groups) * 8 + blockIdx.z * 2 + hh, r = threadIdx.x % kTok;
    float w = 0.f, la = 0.f, decay;
    if (h < p.H && r < live) ssd_gates(p, m0 + r, h, decay, w, la);
    la_s[hh][r] = la;
    __syncthreads();
    ChunkTables* tb = reinterpret_cast<ChunkTables*>(base + lay.gates) + min(h, p.H - 1);
    const bool mine = h < p.H;
    const int a = r >> 4, l = r & 15;
    const float* q = la_s[hh] + a * 16;
    float d = 0.f, g = 0.f;
    for (int i = 0; i < l; ++i)
      if (mine) tb->diag[a][i][l] = 0.f;
    if (mine) tb->diag[a][l][l] = w;
    for (int i = l + 1; i < 16; ++i) {
      d += q[i];
      if (mine) tb->diag[a][i][l] = expf(d) * w;
    }
    for (int i = 0; i <= l; ++i) g += q[i];
    if (mine) tb->row[r] = expf(g);
    if (l == 15) total_s[hh][a] = g;
    __syncthreads();
    if (!mine) return;
    const float* tot = total_s[hh];
    float before = 0.f;
    for (int x = 0; x < a; ++x) before += tot[x];
    tb->start[r] = expf(g + before);
    for (int x = a + 1; x < 4; ++x) {
      if (x > a + 1) d += tot[x - 1];
      tb->col[x - 1][r] = expf(d) * w;
    }
    if (a < 3) d += tot[3];
    tb->end[r] = expf(d) * w;
    return;
  }
  const int i = blockIdx.y * 128 + threadIdx.x;
  if (i >= total) return;
  __nv_bfloat16* dst;
  int col, ch = -1;                                // column inside the tile, channel in q | k | v order (-1: padding)
  if (i < 2 * nk) {
    const int isk = i >= nk ? 1 : 0, k = i - isk * nk, h = k / p.DP;
    col = k - h * p.DP;
    dst = reinterpret_cast<__nv_bfloat16*>(base) + (static_cast<size_t>(h) * 2 + isk) * p.DP * kTok;
    if (col < p.N) ch = (isk * p.HK + h) * p.N + col;
  } else {
    const int k = i - 2 * nk, h = k / (vs * kSlice);
    col = k - h * vs * kSlice;
    dst = reinterpret_cast<__nv_bfloat16*>(base + lay.v) + static_cast<size_t>(h) * vs * kSlice * kTok;
    if (col < p.V) ch = 2 * p.HK * p.N + h * p.V + col;
  }
  const int r0 = blockIdx.z * kRun, rows = ch < 0 ? 0 : min(kRun, live - r0);
  float y[kRun];
#pragma unroll
  for (int r = 0; r < kRun; ++r) y[r] = 0.f;
  if (rows > 0) {
    const int m = m0 + r0, C = ssd_channels(p);
    ssd_inputs<kRun, TAPS>(p, p.hist + static_cast<size_t>(slot) * p.taps * C, ch, m, t0 + r0, p.pos[m], C, rows, y);
  }
#pragma unroll
  for (int r = 0; r < kRun; ++r) dst[tile_at(r0 + r, col)] = __float2bfloat16(y[r]);
}

// Two fp32 values as three bf16 pairs whose sums they are (to 24 bits).
__device__ __forceinline__ void split3(float a, float b, uint32_t (&s)[3]) {
  s[0] = pack2(a, b);
  a -= __uint_as_float(s[0] << 16);
  b -= __uint_as_float(s[0] & 0xffff0000u);
  s[1] = pack2(a, b);
  a -= __uint_as_float(s[1] << 16);
  b -= __uint_as_float(s[1] & 0xffff0000u);
  s[2] = pack2(a, b);
}

// grid (nseq, H, ceil(VP / 64)), 256 threads.  NJ: 64-wide blocks of the key size.
template <int NJ>
__global__ void __launch_bounds__(256, 1) ssd_chunk_scan_kernel(const __grid_constant__ SsdParams p) {
  constexpr int DP = NJ * 64, kKS = DP / 32, kQK = DP * kTok * 2;          // 16-wide key steps of a warp; bytes of a q or k tile
  constexpr uint32_t kV = kTok * kSlice * 2, kStage = 2 * kQK + kV + sizeof(ChunkTables);
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t bars[2];
  pdl_wait();
  const int j = blockIdx.x, h = blockIdx.y;
  const int r0 = p.cu_rows[j], n = p.cu_rows[j + 1] - r0;
  if (n <= 0) return;
  const int slot = ssd_slot(p, j);
  if (slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wv = warp & 3, hn = warp >> 2;
  const int chunks = (n + kTok - 1) / kTok;
  const uint32_t st0 = (smem_u32(smem_raw) + 1023u) & ~1023u, p_s = st0 + 2 * kStage;      // P: three tiles of 8 KiB
  uint8_t* const gen = smem_raw + (st0 - smem_u32(smem_raw));
  float4* red = reinterpret_cast<float4*>(gen + 2 * kStage + 3 * 8192) + wv * 256 + lane;     // [16 columns][tokens, columns][lane]
  const uint32_t bar = smem_u32(bars);
  const ChunkLayout lay = chunk_layout(p);
  const int vslices = (p.VP + kSlice - 1) / kSlice, hk = h / (p.H / p.HK);
  const uint8_t* src = reinterpret_cast<const uint8_t*>(p.chunk) + static_cast<size_t>(chunk_slot(r0, j)) * lay.bytes;
  auto fetch = [&](int c) {
    const uint32_t dst = st0 + (c & 1) * kStage, b = bar + 8 * (c & 1);
    const uint8_t* s = src + c * lay.bytes;
    mbar_arrive_expect_tx(b, kStage);
    bulk_g2s(dst, s + static_cast<size_t>(hk) * 2 * kQK, 2 * kQK, b);
    bulk_g2s(dst + 2 * kQK, s + lay.v + (static_cast<size_t>(h) * vslices + blockIdx.z) * kV, kV, b);
    bulk_g2s(dst + 2 * kQK + kV, s + lay.gates + static_cast<size_t>(h) * sizeof(ChunkTables), sizeof(ChunkTables), b);
  };
  int issued = 0;
  if (threadIdx.x == 0) {
    mbar_init(bar, 1);
    mbar_init(bar + 8, 1);
    mbar_init_fence();
    for (; issued < min(2, chunks); ++issued) fetch(issued);
  }
  __syncthreads();
  const float skip = p.skip ? p.skip[h] : 0.f;
  // this warp's value columns and state fragments: S[8 keys][column lane / 4 | + 8, keys (lane % 4) 2 + {0, 1}]
  const int v0 = blockIdx.z * kSlice + wv * 16, q2 = (lane & 3) * 2, l4 = lane >> 2;
  const bool on = v0 < p.VP;
  float S[2 * kKS][4];
  float* st = p.state + ((static_cast<size_t>(slot) * p.H + h) * p.VP + v0) * DP + hn * (DP / 2);
#pragma unroll
  for (int t = 0; t < 2 * kKS; ++t)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int v = l4 + half * 8;
      const float2 f = v0 + v < p.VP ? *reinterpret_cast<const float2*>(st + static_cast<size_t>(v) * DP + t * 8 + q2) : make_float2(0.f, 0.f);
      S[t][half * 2] = f.x;
      S[t][half * 2 + 1] = f.y;
    }
  bool ok = true;
  int c = 0;
  for (; c < chunks; ++c) {
    const uint32_t qt = st0 + (c & 1) * kStage, kt = qt + kQK, vt = kt + kQK;
    const ChunkTables& tb = *reinterpret_cast<const ChunkTables*>(gen + (c & 1) * kStage + 2 * kQK + kV);
    ok = __syncthreads_and(mbar_wait(bar + 8 * (c & 1), (c >> 1) & 1, p.err, kErrWaitFull)) != 0;
    if (!ok) break;
    // ---- pair weights: the ten 16 x 16 tiles on and below the diagonal, dealt to the warps
    for (int tile = warp; tile < 10; tile += 8) {
      const int mi = tile >= 6 ? 3 : tile >= 3 ? 2 : tile >= 1 ? 1 : 0, nt = tile - mi * (mi + 1) / 2;
      const int ar = mi * 16 + (lane & 15), br = nt * 16 + ((lane >> 4) << 3) + (lane & 7);
      float s[2][2][4] = {};                       // [even | odd steps]: two chains
#pragma unroll
      for (int ks = 0; ks < 2 * kKS; ++ks) {
        uint32_t a[4], b[4];
        const int ac = ks * 2 + (lane >> 4), bc = ks * 2 + ((lane >> 3) & 1);
        ldsm4(a, qt + (ac >> 3) * 8192 + ar * 128 + (((ac ^ ar) & 7) << 4));
        ldsm4(b, kt + (bc >> 3) * 8192 + br * 128 + (((bc ^ br) & 7) << 4));
        mma16816(s[ks & 1][0], a, b[0], b[1]);
        mma16816(s[ks & 1][1], a, b[2], b[3]);
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int il = l4 + half * 8, i = mi * 16 + il;
        const float ri = tb.row[i];
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          const int jl = t * 8 + q2, jc = nt * 16 + jl;
          float2 f;
          if (nt == mi) {
            f = *reinterpret_cast<const float2*>(&tb.diag[mi][il][jl]);
          } else {
            f = *reinterpret_cast<const float2*>(&tb.col[mi - 1][jc]);
            f.x *= ri;
            f.y *= ri;
          }
          float x = (s[0][t][half * 2] + s[1][t][half * 2]) * f.x, y = (s[0][t][half * 2 + 1] + s[1][t][half * 2 + 1]) * f.y;
          if (nt == mi) {
            if (il == jl) x += skip;
            if (il == jl + 1) y += skip;
          }
          uint32_t sp[3];
          split3(x, y, sp);
#pragma unroll
          for (int e = 0; e < 3; ++e)
            asm volatile("st.shared.b32 [%0], %1;" ::"r"(p_s + e * 8192 + i * 128 + ((((jc >> 3) ^ i) & 7) << 4) + q2 * 2), "r"(sp[e]) : "memory");
        }
      }
    }
    // ---- read-out of the state at the chunk's start, this warp's half of the keys
    float o[4][2][4] = {};
    if (on) {
#pragma unroll
      for (int ks = 0; ks < kKS; ++ks) {
        uint32_t b[2][2][3];                       // [8 columns][8 keys][part]
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          split3(S[2 * ks][2 * t], S[2 * ks][2 * t + 1], b[t][0]);
          split3(S[2 * ks + 1][2 * t], S[2 * ks + 1][2 * t + 1], b[t][1]);
        }
        uint32_t a[4][4];
#pragma unroll
        for (int mt = 0; mt < 4; ++mt) {
          const int ar = mt * 16 + (lane & 15), ac = (hn * kKS + ks) * 2 + (lane >> 4);
          ldsm4(a[mt], qt + (ac >> 3) * 8192 + ar * 128 + (((ac ^ ar) & 7) << 4));
        }
#pragma unroll
        for (int e = 2; e >= 0; --e)
#pragma unroll
          for (int mt = 0; mt < 4; ++mt)
#pragma unroll
            for (int t = 0; t < 2; ++t) mma16816(o[mt][t], a[mt], b[t][0][e], b[t][1][e]);
      }
#pragma unroll
      for (int mt = 0; mt < 4; ++mt) {
        const float s0 = tb.start[mt * 16 + l4], s1 = tb.start[mt * 16 + l4 + 8];
#pragma unroll
        for (int t = 0; t < 2; ++t) { o[mt][t][0] *= s0; o[mt][t][1] *= s0; o[mt][t][2] *= s1; o[mt][t][3] *= s1; }
      }
    }
    __syncthreads();                               // every warp's pair weights are in place
    if (on) {
      // ---- products inside the chunk: sixteens 0 and 3 of the keys by one half, 1 and 2 by the other
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int ks = u == 0 ? hn : 3 - hn;
        uint32_t b[4];
        const int br = ks * 16 + (lane & 15), bc = wv * 2 + (lane >> 4);
        ldsm4_t(b, vt + br * 128 + (((bc ^ br) & 7) << 4));
#pragma unroll
        for (int mt = 0; mt < 4; ++mt) {
          if (mt < ks) continue;                   // (uniform)
          const int ar = mt * 16 + (lane & 15), ac = ks * 2 + (lane >> 4);
#pragma unroll
          for (int e = 2; e >= 0; --e) {
            uint32_t a[4];
            ldsm4(a, p_s + e * 8192 + ar * 128 + (((ac ^ ar) & 7) << 4));
            mma16816(o[mt][0], a, b[0], b[1]);
            mma16816(o[mt][1], a, b[2], b[3]);
          }
        }
      }
      if (hn == 1) {
#pragma unroll
        for (int mt = 0; mt < 4; ++mt)
#pragma unroll
          for (int t = 0; t < 2; ++t) red[(mt * 2 + t) * 32] = make_float4(o[mt][t][0], o[mt][t][1], o[mt][t][2], o[mt][t][3]);
      }
      // ---- state at the chunk's end
      const float at = tb.start[kTok - 1];
#pragma unroll
      for (int t = 0; t < 2 * kKS; ++t) { S[t][0] *= at; S[t][1] *= at; S[t][2] *= at; S[t][3] *= at; }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        uint32_t vr[4], a[3][4];
        {
          const int r = ks * 16 + (lane & 7) + ((lane >> 4) << 3), vc = wv * 2 + ((lane >> 3) & 1);
          ldsm4_t(vr, vt + r * 128 + (((vc ^ r) & 7) << 4));
        }
        const float2 e0 = *reinterpret_cast<const float2*>(&tb.end[ks * 16 + q2]), e8 = *reinterpret_cast<const float2*>(&tb.end[ks * 16 + q2 + 8]);
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          uint32_t sp[3];
          split3(__uint_as_float(vr[x] << 16) * (x < 2 ? e0.x : e8.x), __uint_as_float(vr[x] & 0xffff0000u) * (x < 2 ? e0.y : e8.y), sp);
          a[0][x] = sp[0];
          a[1][x] = sp[1];
          a[2][x] = sp[2];
        }
#pragma unroll
        for (int nt = 0; nt < kKS; ++nt) {
          uint32_t b[4];
          const int r = ks * 16 + (lane & 15), kc = (hn * kKS + nt) * 2 + (lane >> 4);
          ldsm4_t(b, kt + (kc >> 3) * 8192 + r * 128 + (((kc ^ r) & 7) << 4));
#pragma unroll
          for (int e = 2; e >= 0; --e) {
            mma16816(S[2 * nt], a[e], b[0], b[1]);
            mma16816(S[2 * nt + 1], a[e], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();                               // the stage and the pair weights are free, the second halves in place
    if (threadIdx.x == 0 && c + 2 < chunks) { fetch(c + 2); ++issued; }
    if (on && hn == 0) {
      const int live = n - c * kTok;
      float* out = p.o + (static_cast<size_t>(r0 + c * kTok) * p.H + h) * p.VP + v0;
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          const float4 x = red[(mt * 2 + t) * 32];
          if (v0 + t * 8 >= p.VP) continue;
          const int i = mt * 16 + l4;
          float* d = out + static_cast<size_t>(i) * p.H * p.VP + t * 8 + q2;
          if (i < live) *reinterpret_cast<float2*>(d) = make_float2(o[mt][t][0] + x.x, o[mt][t][1] + x.y);
          if (i + 8 < live)
            *reinterpret_cast<float2*>(d + static_cast<size_t>(8) * p.H * p.VP) = make_float2(o[mt][t][2] + x.z, o[mt][t][3] + x.w);
        }
    }
  }
  if (!ok && threadIdx.x == 0)                                      // do not leave while an own copy is in flight
    for (int i = c; i < issued; ++i) mbar_wait(bar + 8 * (i & 1), (i >> 1) & 1, p.err, kErrWaitDrain);
  if (!ok) return;
#pragma unroll
  for (int t = 0; t < 2 * kKS; ++t)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int v = l4 + half * 8;
      if (v0 + v < p.VP) *reinterpret_cast<float2*>(st + static_cast<size_t>(v) * DP + t * 8 + q2) = make_float2(S[t][half * 2], S[t][half * 2 + 1]);
    }
}

template <int NJ>
static int chunk_go(const SsdParams& p, cudaStream_t stream) {
  constexpr int smem = 2 * (2 * NJ * 64 * kTok * 2 + kTok * kSlice * 2 + static_cast<int>(sizeof(ChunkTables))) + 3 * 8192 + 4 * 4096 + 1024;
  static bool ready[64];
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return static_cast<int>(cudaErrorInvalidDevice);
  if (!ready[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(ssd_chunk_scan_kernel<NJ>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    ready[dev] = true;
  }
  const int vs = (p.VP + kSlice - 1) / kSlice, channels = 2 * p.HK * p.DP + p.H * vs * kSlice;
  const dim3 grid(p.M / kTok + p.nseq, (channels + 127) / 128 + (p.H + 7) / 8, kTok / kRun);
  const cudaError_t e = p.taps == 4   ? launch(ssd_chunk_prep_kernel<4>, grid, dim3(128), 0, stream, 0, p)
                        : p.taps == 0 ? launch(ssd_chunk_prep_kernel<-1>, grid, dim3(128), 0, stream, 0, p)
                                      : launch(ssd_chunk_prep_kernel<0>, grid, dim3(128), 0, stream, 0, p);
  if (e != cudaSuccess) return static_cast<int>(e);
  return static_cast<int>(launch(ssd_chunk_scan_kernel<NJ>, dim3(p.nseq, p.H, vs), dim3(256), smem, stream, 0, p));
}

}  // namespace saber

extern "C" size_t saber_ssd_chunk_floats(const saber::SsdParams* p) {
  if (p->DP > 256 || (p->DP & 63)) return 0;
  return (static_cast<size_t>(p->M) / saber::kTok + p->nseq) * saber::chunk_layout(*p).bytes / 4;
}
int saber_ssd_chunk_launches() { return 2; }
int saber_ssd_chunk_launch(const saber::SsdParams* p, cudaStream_t stream) {
  switch (p->DP) {
    case 64: return saber::chunk_go<1>(*p, stream);
    case 128: return saber::chunk_go<2>(*p, stream);
    case 192: return saber::chunk_go<3>(*p, stream);
    case 256: return saber::chunk_go<4>(*p, stream);
    default: return static_cast<int>(cudaErrorInvalidValue);
  }
}
