// Kernels around the two products of a parallel layer, x <- x + (mixer(h) + ff(h)) with h = tanh(alpha x) w + b:
//
//   residual_tanh   a = x + y + bias (each optional), fp32; stores a and either tanh(alpha a) w + b or a itself in the
//                   activation type (the operand of the next product), the latter also into columns of a wider row
//   gated_norm      mixer outputs in equal groups, each divided by its root mean square, times a weight, gated by a
//                   sigmoid or silu of another projection before or after the norm
//
// Everything here is 32-bit between the loads and the stores; the file is compiled without fast-math (tanh).
#include "ptx.cuh"
#include "launch.cuh"
#include "vec.cuh"
#include <math.h>

namespace skein {

struct ResidualTanhParams {
  const float* x;            // [T, C] or null
  const void* y;             // [T, C] fp32 (y_f32) or activation type, or null
  const float* bias;         // [C] or null
  const float* alpha;        // [1], or null: act_out is a itself
  const float* w;            // [C]
  const float* b;            // [C]
  float* x_out;              // [T, C] or null
  void* act_out;             // [T, act_ld] activation type, or null
  long long act_ld;
  int T, C, y_f32;
};

// tanh with an error of a few units in the last place of fp32, cheaper than the library call for large arguments
__device__ __forceinline__ float tanh_f(float z) {
  const float a = fabsf(z);
  if (a < 0.625f) return tanhf(z);
  const float e = expf(-2.f * a);            // (0, 0.29]
  return copysignf((1.f - e) / (1.f + e), z);
}

template <typename T, int V>
__global__ void __launch_bounds__(256) residual_tanh_kernel(const ResidualTanhParams p) {
  pdl_trigger();
  pdl_wait();
  const int per_row = p.C / V;
  const long long n = (long long)p.T * per_row;
  const float alpha = p.alpha ? p.alpha[0] : 0.f;
  for (long long j = (long long)blockIdx.x * blockDim.x + threadIdx.x; j < n; j += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(j / per_row), c = (int)(j % per_row) * V;
    const size_t i = (size_t)t * p.C + c;
    float a[V];
#pragma unroll
    for (int k = 0; k < V; ++k) a[k] = 0.f;
    if (p.x) load_v<float, V>(p.x + i, a);
    if (p.y) {
      float v[V];
      if (p.y_f32) load_v<float, V>((const float*)p.y + i, v);
      else load_v<T, V>((const T*)p.y + i, v);
#pragma unroll
      for (int k = 0; k < V; ++k) a[k] += v[k];
    }
    if (p.bias) {
      float v[V];
      load_v<float, V>(p.bias + c, v);
#pragma unroll
      for (int k = 0; k < V; ++k) a[k] += v[k];
    }
    if (p.x_out) store_v<float, V>(p.x_out + i, a);
    if (!p.act_out) continue;
    if (p.alpha) {
      float w[V], b[V];
      load_v<float, V>(p.w + c, w);
      load_v<float, V>(p.b + c, b);
#pragma unroll
      for (int k = 0; k < V; ++k) a[k] = tanh_f(alpha * a[k]) * w[k] + b[k];
    }
    store_v<T, V>((T*)p.act_out + (size_t)t * p.act_ld + c, a);
  }
}

struct GatedNormParams {
  const void* o;             // [T, n] activation type
  const void* gate;          // [T, gate_ld] activation type
  const float* w;            // [w_period], or of every column when w_period == n
  void* out;                 // [T, out_ld]
  long long gate_ld, out_ld;
  int T, n, groups, w_period;
  int gate_first;            // the gate multiplies before the norm
  int silu;                  // gate activation: silu, else sigmoid
  float eps, scale;
};

template <typename T>
__device__ __forceinline__ float gate_value(const GatedNormParams& p, float z) {
  const float s = 1.f / (1.f + expf(-z));
  return p.silu ? z * s : s;
}

// TPG threads per group (a warp, or the whole CTA); V elements per access
template <typename T, int V, bool WARP>
__global__ void __launch_bounds__(256) gated_norm_kernel(const GatedNormParams p) {
  __shared__ float sh[8];
  pdl_trigger();
  pdl_wait();
  const int size = p.n / p.groups;
  const int lane = WARP ? threadIdx.x & 31 : threadIdx.x, tpg = WARP ? 32 : blockDim.x;
  const long long u = WARP ? (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.x;
  if (u >= (long long)p.T * p.groups) return;      // (whole warps or the whole CTA)
  const int t = (int)(u / p.groups), c0 = (int)(u % p.groups) * size;
  const T* o = (const T*)p.o + (size_t)t * p.n + c0;
  const T* g = (const T*)p.gate + (size_t)t * p.gate_ld + c0;
  T* out = (T*)p.out + (size_t)t * p.out_ld + c0;
  float ss = 0.f;
  for (int i = lane * V; i < size; i += tpg * V) {
    float v[V], z[V];
    load_v<T, V>(o + i, v);
    if (p.gate_first) {
      load_v<T, V>(g + i, z);
#pragma unroll
      for (int k = 0; k < V; ++k) v[k] *= gate_value<T>(p, z[k]);
    }
#pragma unroll
    for (int k = 0; k < V; ++k) ss += v[k] * v[k];
  }
  for (int k = 16; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
  if (!WARP) {
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
    for (int k = 0; k < (int)(blockDim.x >> 5); ++k) ss += sh[k];
  }
  const float r = p.scale / sqrtf(ss / (float)size + p.eps);
  for (int i = lane * V; i < size; i += tpg * V) {
    float v[V], z[V], w[V];
    load_v<T, V>(o + i, v);
    load_v<T, V>(g + i, z);
    load_v<float, V>(p.w + (c0 + i) % p.w_period, w);
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] *= gate_value<T>(p, z[k]) * r * w[k];
    store_v<T, V>(out + i, v);
  }
}

// The same for groups of up to 4096 elements, four of a group in each thread: read once, kept in registers. A warp per group (WARP), or
// a CTA of the group's size / 4 threads.
template <typename T, bool WARP>
__global__ void __launch_bounds__(1024) gated_norm_reg_kernel(const GatedNormParams p) {
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  const int size = p.n / p.groups, lane = WARP ? threadIdx.x & 31 : threadIdx.x;
  const long long u = WARP ? (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.x;
  if (u >= (long long)p.T * p.groups) return;      // (whole warps or the whole CTA)
  const int t = (int)(u / p.groups), c0 = (int)(u % p.groups) * size, i = lane * 4;
  const bool in = i < size;
  float v[4] = {0.f, 0.f, 0.f, 0.f}, z[4] = {0.f, 0.f, 0.f, 0.f}, w[4] = {0.f, 0.f, 0.f, 0.f}, ss = 0.f;
  if (in) {
    load_v<T, 4>((const T*)p.o + (size_t)t * p.n + c0 + i, v);
    load_v<T, 4>((const T*)p.gate + (size_t)t * p.gate_ld + c0 + i, z);
    load_v<float, 4>(p.w + (c0 + i) % p.w_period, w);
  }
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    z[k] = gate_value<T>(p, z[k]);
    if (p.gate_first) v[k] *= z[k];
    ss += v[k] * v[k];
  }
  for (int k = 16; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
  if (!WARP) {
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
    for (int k = 0; k < (int)(blockDim.x >> 5); ++k) ss += sh[k];
  }
  if (!in) return;
  const float r = p.scale / sqrtf(ss / (float)size + p.eps);
#pragma unroll
  for (int k = 0; k < 4; ++k) v[k] *= p.gate_first ? r * w[k] : z[k] * r * w[k];
  store_v<T, 4>((T*)p.out + (size_t)t * p.out_ld + c0 + i, v);
}

}  // namespace skein

extern "C" int skein_residual_tanh(const float* x, const void* y, int y_f32, const float* bias, const float* alpha, const float* w, const float* b,
                                   float* x_out, void* act_out, long long act_ld, int T, int C, int fp32, void* stream) {
  using namespace skein;
  if (T == 0 || C == 0) return 0;
  ResidualTanhParams p{x, y, bias, alpha, w, b, x_out, act_out, act_ld, T, C, y_f32};
  const bool v4 = C % 4 == 0 && act_ld % 4 == 0 && ((uintptr_t)act_out % 16) == 0;
  const long long n = (long long)T * C / (v4 ? 4 : 1);
  const long long want = (n + 255) / 256;
  const dim3 grid((unsigned)(want > 148 * 16 ? 148 * 16 : want));
  cudaStream_t s = (cudaStream_t)stream;
  if (fp32) return (int)(v4 ? launch_pdl(residual_tanh_kernel<float, 4>, grid, dim3(256), 0, s, p) : launch_pdl(residual_tanh_kernel<float, 1>, grid, dim3(256), 0, s, p));
  return (int)(v4 ? launch_pdl(residual_tanh_kernel<__nv_bfloat16, 4>, grid, dim3(256), 0, s, p)
                  : launch_pdl(residual_tanh_kernel<__nv_bfloat16, 1>, grid, dim3(256), 0, s, p));
}

// groups divides n; w_period divides the group size or is n.
extern "C" int skein_gated_norm(const void* o, const void* gate, long long gate_ld, const float* w, int w_period, void* out, long long out_ld, int T,
                                int n, int groups, int gate_first, int silu, float eps, float scale, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (groups < 1 || n % groups != 0 || (w_period != n && (n / groups) % w_period != 0)) return -1;
  GatedNormParams p{o, gate, w, out, gate_ld, out_ld, T, n, groups, w_period, gate_first, silu, eps, scale};
  const int size = n / groups;
  const bool v4 = size % 4 == 0 && w_period % 4 == 0 && gate_ld % 4 == 0 && out_ld % 4 == 0 && (uintptr_t)gate % 16 == 0 && (uintptr_t)out % 16 == 0 &&
                  (uintptr_t)o % 16 == 0;
  const bool warp = size <= 512;
  const long long units = (long long)T * groups;
  const dim3 grid((unsigned)(warp ? (units + 7) / 8 : units));
  cudaStream_t s = (cudaStream_t)stream;
  if (v4 && size <= 4096) {
    const bool w32 = size <= 128;
    const dim3 g((unsigned)(w32 ? (units + 7) / 8 : units)), b(w32 ? 256 : (size / 4 + 31) / 32 * 32);
    if (fp32) return (int)(w32 ? launch_pdl(gated_norm_reg_kernel<float, true>, g, b, 0, s, p) : launch_pdl(gated_norm_reg_kernel<float, false>, g, b, 0, s, p));
    return (int)(w32 ? launch_pdl(gated_norm_reg_kernel<__nv_bfloat16, true>, g, b, 0, s, p)
                     : launch_pdl(gated_norm_reg_kernel<__nv_bfloat16, false>, g, b, 0, s, p));
  }
  auto go = [&](auto fn) -> int { return (int)launch_pdl(fn, grid, dim3(256), 0, s, p); };
  if (fp32) {
    if (v4) return warp ? go(gated_norm_kernel<float, 4, true>) : go(gated_norm_kernel<float, 4, false>);
    return warp ? go(gated_norm_kernel<float, 1, true>) : go(gated_norm_kernel<float, 1, false>);
  }
  if (v4) return warp ? go(gated_norm_kernel<__nv_bfloat16, 4, true>) : go(gated_norm_kernel<__nv_bfloat16, 4, false>);
  return warp ? go(gated_norm_kernel<__nv_bfloat16, 1, true>) : go(gated_norm_kernel<__nv_bfloat16, 1, false>);
}
