// Plain tiled GEMM on the FMA pipes: Y[t, f] = sum_k X[t, k] * W[f, k], accumulated in fp32.
//
// It covers what the tensor-core kernel (gemm_ws.cu) does not take: true 32-bit products (a model run in fp32) and bf16
// operands whose row length is not a multiple of 8 elements. Same forms as there: one matrix, one matrix per expert over
// ragged row lists whose sizes live in device memory, or one matrix per head over column blocks of the same rows; the same
// epilogues (gate/up activation, multiplication by a sigmoid gate). 64 x 64 output tile, 16-wide K steps, 4 x 4 outputs per
// thread.
#include "gemm_sched.cuh"
#include "launch.cuh"
#include <cuda_bf16.h>

namespace skein {

constexpr int GS_TILE = 64, GS_K = 16;

template <typename T> __device__ __forceinline__ float gs_load(const void* p, size_t i);
template <> __device__ __forceinline__ float gs_load<float>(const void* p, size_t i) { return ((const float*)p)[i]; }
template <> __device__ __forceinline__ float gs_load<__nv_bfloat16>(const void* p, size_t i) { return __bfloat162float(((const __nv_bfloat16*)p)[i]); }

// grid = (feature tiles, row tiles, groups), 256 threads
template <typename T, bool DUAL>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const SkeinGemmParams p) {
  __shared__ float ws[DUAL ? 2 : 1][GS_K][GS_TILE + 4];
  __shared__ float xs[GS_K][GS_TILE + 4];
  pdl_trigger();
  pdl_wait();
  const int g = blockIdx.z, f0 = blockIdx.x * GS_TILE, t0 = blockIdx.y * GS_TILE;
  const int cnt = p.group_cnt ? p.group_cnt[g] : p.t_static;
  const int off = p.group_off ? p.group_off[g] : 0;
  if (t0 >= cnt) return;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const size_t ldx = p.x_ld > 0 ? p.x_ld : p.K;
  const size_t wrow0 = (size_t)g * p.w_rows_per_group;
  float acc[DUAL ? 2 : 1][4][4];
#pragma unroll
  for (int d = 0; d < (DUAL ? 2 : 1); ++d)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[d][i][j] = 0.f;
  for (int k0 = 0; k0 < p.K; k0 += GS_K) {
    for (int i = tid; i < GS_TILE * GS_K; i += 256) {
      const int r = i / GS_K, k = i % GS_K;
      const bool kin = k0 + k < p.K;
      xs[k][r] = (kin && t0 + r < cnt) ? gs_load<T>(p.X, (size_t)(off + t0 + r) * ldx + (size_t)g * p.x_group_cols + k0 + k) : 0.f;
#pragma unroll
      for (int d = 0; d < (DUAL ? 2 : 1); ++d)
        ws[d][k][r] = (kin && f0 + r < p.F) ? gs_load<T>(p.W, (wrow0 + (d ? p.up_row_off : 0) + f0 + r) * (size_t)p.K + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GS_K; ++k) {
      float xv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) xv[i] = xs[k][ty * 4 + i];
#pragma unroll
      for (int d = 0; d < (DUAL ? 2 : 1); ++d) {
        float wv[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) wv[j] = ws[d][k][tx * 4 + j];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[d][i][j] = fmaf(xv[i], wv[j], acc[d][i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + ty * 4 + i;
    if (t >= cnt) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int f = f0 + tx * 4 + j;
      if (f >= p.F) continue;
      float y = acc[0][i][j];
      if (DUAL) y = glu_act(p, y, acc[DUAL ? 1 : 0][i][j]);
      const size_t row = (size_t)(off + t), gcol = (size_t)g * p.out_group_cols + f;
      if (p.gate) y *= sigmoid_f(gs_load<T>(p.gate, row * p.gate_ld + gcol));
      const size_t idx = row * p.ldo + p.out_col0 + gcol;
      if (f < p.relu2_cols) y = relu2(y);
      if (p.residual) y += p.out_f32 ? gs_load<float>(p.residual, idx) : gs_load<T>(p.residual, idx);
      if (p.out_f32 || sizeof(T) == 4) ((float*)p.out)[idx] = y;
      else ((__nv_bfloat16*)p.out)[idx] = __float2bfloat16(y);
    }
  }
}

}  // namespace skein

// max_rows bounds the rows of any group (a host-side bound: the true counts may live on the device).
extern "C" int skein_gemm_simt(const SkeinGemmParams* p, int fp32, int max_rows, void* stream) {
  using namespace skein;
  if (!p || p->G < 1 || p->G > 65535 || p->K < 1 || p->F < 1 || (p->mode != 0 && p->mode != 1)) return -1;
  if (max_rows <= 0) return 0;
  const dim3 grid((p->F + GS_TILE - 1) / GS_TILE, (max_rows + GS_TILE - 1) / GS_TILE, p->G);
  cudaStream_t s = (cudaStream_t)stream;
  if (fp32) return (int)(p->mode == 1 ? launch_pdl(gemm_simt_kernel<float, true>, grid, dim3(256), 0, s, *p)
                                      : launch_pdl(gemm_simt_kernel<float, false>, grid, dim3(256), 0, s, *p));
  return (int)(p->mode == 1 ? launch_pdl(gemm_simt_kernel<__nv_bfloat16, true>, grid, dim3(256), 0, s, *p)
                            : launch_pdl(gemm_simt_kernel<__nv_bfloat16, false>, grid, dim3(256), 0, s, *p));
}
