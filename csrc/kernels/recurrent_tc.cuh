// Shared by the tensor-core forms of the recurrences (recurrent_tc.cu, recurrent_channel_tc.cu): chunks of 64 tokens, values as a sum of two
// bf16 numbers (hi + lo, 16 bits of mantissa), and the inverse of a chunk's unit lower triangular matrix.
#pragma once
#include "ptx.cuh"
#include <cuda_bf16.h>
#include <stdint.h>

namespace skein {

constexpr int RT_C = 64;                       // tokens of a chunk
constexpr int RT_MAT_BYTES = RT_C * RT_C * 2;
constexpr uint64_t RT_BUDGET_NS = 4000000000ull;

// Chunks of sequence s are numbered from q_start / 64 + s: sequences lie one after another, so the ranges do not meet.
__device__ __forceinline__ int rt_chunk0(int q_start, int seq) { return q_start / RT_C + seq; }

__device__ __forceinline__ uint32_t rt_pack(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}
// a + b ~ hi + lo with both bf16 pairs
__device__ __forceinline__ void rt_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = rt_pack(a - f.x, b - f.y);
}

__device__ __forceinline__ void rt_ldsm4(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void rt_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ void rt_ldsm2t(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}

constexpr int RT_LX = RT_C + 8, RT_LY = 40, RT_LD = 20;    // row lengths of the 64-wide and 32-wide bf16 and the 16-wide fp32 scratch matrices

// One 16 x 8 tile of L R with both factors as hi + lo: acc over `ks` steps of 16. l, r: shared-memory addresses of the tile's
// rows in the hi parts; the lo parts lie l_lo, r_lo bytes further.
__device__ __forceinline__ void rt_tile(float* acc, uint32_t l, uint32_t l_lo, int l_ld, uint32_t r, uint32_t r_lo, int r_ld, int ks) {
  const int lane = threadIdx.x & 31;
  acc[0] = acc[1] = acc[2] = acc[3] = 0.f;
  for (int k = 0; k < ks; ++k) {
    uint32_t ah[4], al[4], bh[2], bl[2];
    const uint32_t la = l + ((lane & 15) * l_ld + k * 16 + (lane >> 4) * 8) * 2, ra = r + (k * 16 + (lane & 15)) * r_ld * 2;
    rt_ldsm4(la, ah);
    rt_ldsm4(la + l_lo, al);
    rt_ldsm2t(ra, bh);
    rt_ldsm2t(ra + r_lo, bl);
    rt_mma(acc, ah, bh[0], bh[1]);
    rt_mma(acc, al, bh[0], bh[1]);
    rt_mma(acc, ah, bl[0], bl[1]);
  }
}

// a tile's accumulators, negated or not, as hi + lo into a bf16 scratch matrix
__device__ __forceinline__ void rt_put_tile(const float* acc, float sign, __nv_bfloat16* hi, __nv_bfloat16* lo, int ld) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    uint32_t h, l;
    rt_split(sign * acc[2 * e], sign * acc[2 * e + 1], h, l);
    const int at = ((lane >> 2) + 8 * e) * ld + (lane & 3) * 2;
    *reinterpret_cast<uint32_t*>(hi + at) = h;
    *reinterpret_cast<uint32_t*>(lo + at) = l;
  }
}

// X = (I + A)^-1 of a strictly lower triangular A [64, 64]: the 16 x 16 blocks on the diagonal by substitution, then blocks of 32 and 64 from
// two of half the size, [[a, 0], [b, d]]^-1 = [[a^-1, 0], [-d^-1 b a^-1, d^-1]]. A is given by its diagonal blocks Ad [64][RT_LD] fp32 and the
// blocks below them as hi + lo [64][RT_LX]; X comes as hi + lo [64][RT_LX] (the lo parts right behind the hi parts); Yh, Yl [32][RT_LY] are scratch. 256 threads;
// A must be complete (a barrier ahead of the call), X is at the return.
__device__ __forceinline__ void rt_invert(const float* Ad, const __nv_bfloat16* Ah, __nv_bfloat16* Xh, __nv_bfloat16* Xl, __nv_bfloat16* Yh, __nv_bfloat16* Yl) {
  const int tid = threadIdx.x, warp = tid >> 5;
  for (int i = tid; i < 2 * RT_C * RT_LX / 8; i += 256) reinterpret_cast<uint4*>(Xh)[i] = make_uint4(0, 0, 0, 0);
  __syncthreads();
  if (tid < RT_C) {
    const int b0 = tid & ~15, col = tid & 15;
    float x[16];
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      float s = r == col ? 1.f : 0.f;
#pragma unroll
      for (int m = 0; m < r; m += 4) {
        const float4 a = *reinterpret_cast<const float4*>(Ad + (b0 + r) * RT_LD + m);
        s = fmaf(-a.x, x[m], s);
        if (m + 1 < r) s = fmaf(-a.y, x[m + 1], s);
        if (m + 2 < r) s = fmaf(-a.z, x[m + 2], s);
        if (m + 3 < r) s = fmaf(-a.w, x[m + 3], s);
      }
      x[r] = s;
    }
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      const __nv_bfloat16 hi = __float2bfloat16(x[r]);
      Xh[(b0 + r) * RT_LX + b0 + col] = hi;
      Xl[(b0 + r) * RT_LX + b0 + col] = __float2bfloat16(x[r] - __bfloat162float(hi));
    }
  }
  __syncthreads();
  constexpr uint32_t X_LO = RT_C * RT_LX * 2, Y_LO = 32 * RT_LY * 2;
  const uint32_t xa = smem_u32(Xh), aa = smem_u32(Ah), ya = smem_u32(Yh);
  auto x_at = [&](int r, int q) { return xa + (r * RT_LX + q) * 2; };
  float acc[4];
  const int b16 = 32 * (warp >> 1), q16 = 8 * (warp & 1);              // blocks of 32: a warp per 16 x 8 tile
  if (warp < 4) {
    rt_tile(acc, aa + ((b16 + 16) * RT_LX + b16) * 2, X_LO, RT_LX, x_at(b16, b16 + q16), X_LO, RT_LX, 1);
    rt_put_tile(acc, 1.f, Yh + (b16 / 2) * RT_LY + q16, Yl + (b16 / 2) * RT_LY + q16, RT_LY);
  }
  __syncthreads();
  if (warp < 4) {
    rt_tile(acc, x_at(b16 + 16, b16 + 16), X_LO, RT_LX, ya + ((b16 / 2) * RT_LY + q16) * 2, Y_LO, RT_LY, 1);
    rt_put_tile(acc, -1.f, Xh + (b16 + 16) * RT_LX + b16 + q16, Xl + (b16 + 16) * RT_LX + b16 + q16, RT_LX);
  }
  __syncthreads();
  const int r32 = 16 * (warp >> 2), q32 = 8 * (warp & 3);              // the block of 64
  rt_tile(acc, aa + ((32 + r32) * RT_LX) * 2, X_LO, RT_LX, x_at(0, q32), X_LO, RT_LX, 2);
  rt_put_tile(acc, 1.f, Yh + r32 * RT_LY + q32, Yl + r32 * RT_LY + q32, RT_LY);
  __syncthreads();
  rt_tile(acc, x_at(32 + r32, 32), X_LO, RT_LX, ya + q32 * 2, Y_LO, RT_LY, 2);
  rt_put_tile(acc, -1.f, Xh + (32 + r32) * RT_LX + q32, Xl + (32 + r32) * RT_LX + q32, RT_LX);
  __syncthreads();
}

}  // namespace skein
