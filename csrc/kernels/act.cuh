// Activations behind projections and convolutions, for files compiled without fast-math.
#pragma once
#include <cuda_bf16.h>
#include <math.h>

namespace skein {

// silu; where the result is rounded to bf16 it is computed fast
template <typename T> __device__ __forceinline__ float silu_act(float z);
template <> __device__ __forceinline__ float silu_act<float>(float z) { return z / (1.f + expf(-z)); }
template <> __device__ __forceinline__ float silu_act<__nv_bfloat16>(float z) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(z * -1.44269504f));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
  return z * r;
}
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// The same in about half the instructions: log(1 + e) = 2 atanh(e / (2 + e)) by its series, whose argument is at most 1/3 (seven terms leave
// 1e-8). Relative error below 1e-6 down to z = -16.
__device__ __forceinline__ float softplus_series(float z) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(fabsf(z) * -1.44269504f));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(2.f + e));
  const float s = e * r, q = s * s;
  float p = fmaf(q, 1.f / 13.f, 1.f / 11.f);
  p = fmaf(q, p, 1.f / 9.f);
  p = fmaf(q, p, 1.f / 7.f);
  p = fmaf(q, p, 1.f / 5.f);
  p = fmaf(q, p, 1.f / 3.f);
  return fmaf(2.f * s, fmaf(q, p, 1.f), fmaxf(z, 0.f));
}

}  // namespace skein
