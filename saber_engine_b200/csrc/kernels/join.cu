// Between two sublayers: the result of one is divided by its root mean square and joins the fp32 stream, the stream's row is normed and,
// ahead of a mixer, blended with the row of the token before.
//
// A CTA owns up to four consecutive rows and computes one more where the row ahead of them belongs to the same sequence, so that no
// CTA waits for another: the stream is read from one buffer and written to another.  The CTA of a sequence's first row reads the
// slot's row (h of the portion before) and then replaces it by h of the portion's last row, which it computes once more if that is
// another CTA's.  A thread keeps to its own columns throughout; only the two sums per row cross threads.
#include "join.h"
#include "launch.cuh"
#include "ptx_sm100.cuh"
#include "scan_records.cuh"

namespace saber {

constexpr int kJoinThreads = 512;
constexpr int kJoinMaxRows = 4;

__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float dot4(float4 a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }

// The sublayer's result at columns c .. c + 3 of row m.
__device__ __forceinline__ float4 join_result(const JoinParams& p, int m, int c) {
  float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
  if (p.y != nullptr) z = *reinterpret_cast<const float4*>(p.y + static_cast<size_t>(m) * p.ldy + c);
  if (p.routed != nullptr)
    for (int k0 = 0; k0 < p.routes; k0 += 4) {      // four rows requested together
      int slot[4];
      float w[4];
      float4 v[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int at = m * p.routes + min(k0 + i, p.routes - 1);
        slot[i] = p.slot_of[at];
        w[i] = p.route_w[at];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const size_t at = static_cast<size_t>(max(slot[i], 0)) * p.ldr + c;
        if (p.routed_f32) {
          v[i] = *reinterpret_cast<const float4*>(static_cast<const float*>(p.routed) + at);
        } else {
          const uint2 u = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p.routed) + at);
          v[i] = make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xFFFF0000u));
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (slot[i] >= 0 && k0 + i < p.routes)
          z = make_float4(fmaf(w[i], v[i].x, z.x), fmaf(w[i], v[i].y, z.y), fmaf(w[i], v[i].z, z.z), fmaf(w[i], v[i].w, z.w));
    }
  return z;
}

// The stream row ahead of the sublayer's result.
__device__ __forceinline__ float4 join_base(const JoinParams& p, int m, int c) {
  if (p.table == nullptr) return *reinterpret_cast<const float4*>(p.x + static_cast<size_t>(m) * p.ldx + c);
  const size_t row = static_cast<size_t>(min(max(p.ids[m], 0), p.vocab - 1)) * p.width;
  float v[4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
    v[i] = c + i >= p.width ? 0.f
           : p.embed_scale * (p.table_f32 ? static_cast<const float*>(p.table)[row + c + i] : __bfloat162float(static_cast<const __nv_bfloat16*>(p.table)[row + c + i]));
  return make_float4(v[0], v[1], v[2], v[3]);
}

// Sums over the CTA of N values at a time; every thread gets them.
template <int N>
__device__ __forceinline__ void join_sums(float (&v)[N], float (*red)[kJoinMaxRows + 1]) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int k = 0; k < N; ++k) v[k] += __shfl_xor_sync(0xffffffffu, v[k], o);
  if (lane == 0)
#pragma unroll
    for (int k = 0; k < N; ++k) red[warp][k] = v[k];
  __syncthreads();
#pragma unroll
  for (int k = 0; k < N; ++k) {
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < kJoinThreads / 32; ++w) s += red[w][k];
    v[k] = s;
  }
}

// h of rows m0 .. m0 + N - 1 (those with their bit in `live`) into buf, N rows of ws floats; rows with their bit in `own` go to x_out.
template <int N>
__device__ __forceinline__ void join_rows(const JoinParams& p, int m0, uint32_t live, uint32_t own, float* buf, int ws, float (*red)[kJoinThreads / 32][kJoinMaxRows + 1]) {
  float sum[N] = {};
  const float inv_w = 1.f / static_cast<float>(p.width);
  const bool sub = p.y != nullptr || p.routed != nullptr;
  if (sub) {
    for (int c = threadIdx.x * 4; c < ws; c += kJoinThreads * 4)
#pragma unroll
      for (int k = 0; k < N; ++k) {
        if (!(live >> k & 1u)) continue;
        const float4 z = join_result(p, m0 + k, c);
        *reinterpret_cast<float4*>(buf + k * ws + c) = z;
        sum[k] += dot4(z);
      }
    join_sums<N>(sum, red[0]);
#pragma unroll
    for (int k = 0; k < N; ++k) sum[k] = p.mult / sqrtf(sum[k] * inv_w + p.eps);
  }
  float sq[N] = {};
  for (int c = threadIdx.x * 4; c < ws; c += kJoinThreads * 4) {
    const float4 st = p.step != nullptr ? *reinterpret_cast<const float4*>(p.step + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 pw = sub ? *reinterpret_cast<const float4*>(p.post_w + c) : st;
#pragma unroll
    for (int k = 0; k < N; ++k) {
      if (!(live >> k & 1u)) continue;
      float4* b = reinterpret_cast<float4*>(buf + k * ws + c);
      float4 v = join_base(p, m0 + k, c);
      if (sub) {
        const float4 z = *b;
        v = make_float4(fmaf(z.x * sum[k], pw.x, v.x), fmaf(z.y * sum[k], pw.y, v.y), fmaf(z.z * sum[k], pw.z, v.z), fmaf(z.w * sum[k], pw.w, v.w));
      }
      if (p.step != nullptr) v = add4(v, st);
      *b = v;
      sq[k] += dot4(v);
      if (own >> k & 1u) *reinterpret_cast<float4*>(p.x_out + static_cast<size_t>(m0 + k) * p.ldx + c) = v;
    }
  }
  join_sums<N>(sq, red[1]);
#pragma unroll
  for (int k = 0; k < N; ++k) sq[k] = 1.f / sqrtf(sq[k] * inv_w + p.eps);
  for (int c = threadIdx.x * 4; c < ws; c += kJoinThreads * 4) {
    const float4 w = *reinterpret_cast<const float4*>(p.norm_w + c);
#pragma unroll
    for (int k = 0; k < N; ++k) {
      if (!(live >> k & 1u)) continue;
      float4* b = reinterpret_cast<float4*>(buf + k * ws + c);
      const float4 v = *b;
      *b = make_float4(v.x * sq[k] * w.x, v.y * sq[k] * w.y, v.z * sq[k] * w.z, v.w * sq[k] * w.w);
    }
  }
}

// grid ceil(M / R), 512 threads; shared memory: R + 2 rows (the row ahead, the own rows, a sequence's last row)
template <int R>
__global__ void __launch_bounds__(kJoinThreads) join_kernel(const __grid_constant__ JoinParams p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float4 sm4[];
  float* buf = reinterpret_cast<float*>(sm4);
  __shared__ float red[4][kJoinThreads / 32][kJoinMaxRows + 1];
  __shared__ int seq_s[R];
  const int m0 = blockIdx.x * R, n = min(R, p.M - m0), ws = (p.width + 3) & ~3;
  const uint32_t own = (1u << n) - 1u;
  if (p.shift == nullptr) {
    join_rows<R>(p, m0, own, own, buf + ws, ws, red);
  } else {
    if (threadIdx.x < n) seq_s[threadIdx.x] = seq_of_row(p.cu_rows, p.nseq, m0 + threadIdx.x);
    __syncthreads();
    const bool ahead = seq_s[0] >= 0 && m0 > p.cu_rows[seq_s[0]];
    join_rows<R + 1>(p, m0 - 1, own << 1 | (ahead ? 1u : 0u), own << 1, buf, ws, red);
  }
#pragma unroll 1
  for (int i = 0; i < n; ++i) {
    const int m = m0 + i;
    const float* h = buf + (i + 1) * ws;
    int kind = 0, slot = -1, last = m;              // 0: as it is, 1: the row ahead, 2: the slot's row, 3: zeros
    if (p.shift != nullptr) {
      const int j = seq_s[i];
      if (j < 0) {
        kind = 3;
      } else if (m > p.cu_rows[j]) {
        kind = 1;
      } else {
        kind = 3;
        slot = p.slots[j];
        if (slot >= p.n_slots) {
          if (threadIdx.x == 0 && p.err) atomicCAS(p.err, 0u, static_cast<uint32_t>(kErrBadIndex));
          slot = -1;
        }
        if (slot >= 0 && p.pos[m] > 0) kind = 2;
        last = p.cu_rows[j + 1] - 1;
      }
    }
    float* st = slot >= 0 ? p.state + static_cast<size_t>(slot) * p.width : nullptr;
    for (int c = threadIdx.x * 4; c < ws; c += kJoinThreads * 4) {
      float4 v = *reinterpret_cast<const float4*>(h + c);
      if (kind != 0) {
        float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
        if (kind == 1) {
          b = *reinterpret_cast<const float4*>(h - ws + c);
        } else if (kind == 2) {
          float t[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) t[e] = c + e < p.width ? st[c + e] : 0.f;
          b = make_float4(t[0], t[1], t[2], t[3]);
        }
        const float4 s = *reinterpret_cast<const float4*>(p.shift + c);
        v = make_float4(fmaf(b.x - v.x, s.x, v.x), fmaf(b.y - v.y, s.y, v.y), fmaf(b.z - v.z, s.z, v.z), fmaf(b.w - v.w, s.w, v.w));
      }
      operand_store4(p.op, m, c, v);
    }
    if (st == nullptr) continue;
    const float* hl = buf + (last - m0 + 1) * ws;
    if (last >= m0 + n) {                           // (uniform: the row of another CTA)
      hl = buf + (R + 1) * ws;
      __syncthreads();                              // (its sums may still be read)
      join_rows<1>(p, last, 1u, 0u, buf + (R + 1) * ws, ws, red + 2);
    }
    for (int c = threadIdx.x * 4; c < ws; c += kJoinThreads * 4)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (c + e < p.width) st[c + e] = hl[c + e];
  }
}

template <int R>
static int join_go(const JoinParams& p, int smem, cudaStream_t stream) {
  static bool ready[64];
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return static_cast<int>(cudaErrorInvalidDevice);
  if (!ready[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(join_kernel<R>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    ready[dev] = true;
  }
  return static_cast<int>(launch(join_kernel<R>, dim3((p.M + R - 1) / R), dim3(kJoinThreads), smem, stream, 2, p));
}

}  // namespace saber

extern "C" int saber_join_launch(const saber::JoinParams* p, cudaStream_t stream) {
  using namespace saber;
  if (p->M <= 0 || p->width <= 0 || (p->ldx & 3) || p->ldx < p->width || (p->y != nullptr && ((p->ldy & 3) || p->ldy < p->width)) ||
      (p->routed != nullptr && ((p->ldr & 7) || p->routes < 1 || p->slot_of == nullptr || p->route_w == nullptr)) ||
      ((p->y != nullptr || p->routed != nullptr) && p->post_w == nullptr) || (p->table == nullptr ? p->x == nullptr : p->ids == nullptr) ||
      p->x_out == nullptr || p->norm_w == nullptr || (p->shift != nullptr && (p->state == nullptr || p->x_out == p->x)))
    return static_cast<int>(cudaErrorInvalidValue);
  const int smem = (p->rows + 2) * ((p->width + 3) & ~3) * 4;
  if (smem > 220 * 1024) return static_cast<int>(cudaErrorInvalidValue);
  switch (p->rows) {
    case 1: return join_go<1>(*p, smem, stream);
    case 2: return join_go<2>(*p, smem, stream);
    case 4: return join_go<4>(*p, smem, stream);
    default: return static_cast<int>(cudaErrorInvalidValue);
  }
}
