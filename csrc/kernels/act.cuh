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

}  // namespace skein
