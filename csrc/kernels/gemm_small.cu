// Products of a decode step whose weights are small: Y[t, f] = sum_k X[t, k] W[f, k] for up to 64 rows per tile, bf16, fp32 sums.
//
// The streaming kernel (gemm_ws.cu) is built for weights of tens of megabytes; below a megabyte or two its set-up and the fix-up of cut
// tiles set the time. Here a tile of 64 rows x 32 features belongs to a cluster of CTAs that share the reduction dimension, and every warp
// of a CTA owns a part of its CTA's share: it copies its own 64 x 64 and 32 x 64 pieces with cp.async (two in flight), multiplies them
// with mma.sync without waiting for anybody, and only the sums meet: over the warps in shared memory, over the CTAs through distributed
// shared memory, each CTA finishing some of the rows, in rank order (the result does not depend on timing).
#include "launch.cuh"
#include "ptx.cuh"
#include <cooperative_groups.h>
#include <cuda_bf16.h>

namespace skein {

constexpr int GL_WARPS = 8, GL_THREADS = 32 * GL_WARPS;
constexpr int GL_ROWS = 64, GL_F = 32, GL_K = 64;                      // a warp's piece
constexpr int GL_X_BYTES = GL_ROWS * GL_K * 2, GL_W_BYTES = GL_F * GL_K * 2, GL_STAGE = GL_X_BYTES + GL_W_BYTES;
constexpr int GL_SUM_LD = GL_F + 2;                                    // floats between rows of a parked sum
constexpr int GL_SMEM = GL_WARPS * 2 * GL_STAGE;
constexpr int GL_MAX_CLUSTER = 8;
static_assert(GL_ROWS * GL_SUM_LD * 4 <= GL_STAGE, "a warp's sums fit its own buffer");

struct GemmSmallParams {
  const __nv_bfloat16* x;    // [T, x_ld]
  const __nv_bfloat16* w;    // [F, K]
  void* out;                 // [T, out_ld] bf16 or fp32
  const void* residual;      // same place and type as out, or null
  long long x_ld, out_ld;
  int T, F, K, out_f32;
  int stages;                // buffers of a warp: 2, or 1 where no warp has more than one piece
};

__device__ __forceinline__ uint32_t gl_swz(int row, int chunk) { return (uint32_t)(row * (GL_K * 2) + ((chunk ^ (row & 7)) << 4)); }
__device__ __forceinline__ void gl_copy(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void gl_ldsm(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void gl_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// grid (cluster, feature tiles, row tiles)
__global__ void __launch_bounds__(GL_THREADS) gemm_small_kernel(const GemmSmallParams p) {
  namespace cg = cooperative_groups;
  extern __shared__ __align__(128) uint8_t gl_smem[];
  pdl_trigger();
  pdl_wait();
  cg::cluster_group cluster = cg::this_cluster();
  const int n_cta = gridDim.x, rank = blockIdx.x, f0 = blockIdx.y * GL_F, t0 = blockIdx.z * GL_ROWS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rows = min(GL_ROWS, p.T - t0), m_tiles = (rows + 15) / 16;
  // pieces of 64 along K, dealt round-robin to the warps of the cluster
  const int warp_bytes = p.stages * GL_STAGE;
  const int pieces = (p.K + GL_K - 1) / GL_K, first = rank * GL_WARPS + warp, hop = n_cta * GL_WARPS;
  const int mine = first < pieces ? (pieces - first + hop - 1) / hop : 0;
  uint8_t* buf = gl_smem + warp * warp_bytes;
  const uint32_t base = smem_u32(buf);
  auto issue = [&](int i) {
    if (i < mine) {
      const int k0 = (first + i * hop) * GL_K;
      const uint32_t xs = base + (i & (p.stages - 1)) * GL_STAGE, ws = xs + GL_X_BYTES;
      const int ch = lane & 7, left = p.K - k0 - ch * 8;                   // a lane's chunk of 8 elements lies inside the row or outside
      const int bytes = left > 0 ? 16 : 0;
      const int kk = left > 0 ? k0 + ch * 8 : 0;
#pragma unroll
      for (int r = lane >> 3; r < GL_ROWS; r += 4) {
        const int t = min(t0 + r, p.T - 1);
        gl_copy(xs + gl_swz(r, ch), p.x + (size_t)t * p.x_ld + kk, r < rows ? bytes : 0);
      }
#pragma unroll
      for (int r = lane >> 3; r < GL_F; r += 4) {
        const int f = min(f0 + r, p.F - 1);
        gl_copy(ws + gl_swz(r, ch), p.w + (size_t)f * p.K + kk, f0 + r < p.F ? bytes : 0);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float acc[4][4][4];
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[m][n][i] = 0.f;
  issue(0);
  issue(1);
  for (int i = 0; i < mine; ++i) {
    asm volatile("cp.async.wait_group %0;" ::"n"(1) : "memory");
    __syncwarp();
    const uint32_t xs = base + (i & (p.stages - 1)) * GL_STAGE, ws = xs + GL_X_BYTES;
#pragma unroll
    for (int k = 0; k < GL_K / 16; ++k) {
      uint32_t b[2][4];
      const int mat = lane >> 3;
#pragma unroll
      for (int n = 0; n < 2; ++n) gl_ldsm(ws + gl_swz(n * 16 + (mat >> 1) * 8 + (lane & 7), k * 2 + (mat & 1)), b[n]);
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        if (m >= m_tiles) break;
        uint32_t a[4];
        gl_ldsm(xs + gl_swz(m * 16 + (lane & 15), k * 2 + (lane >> 4)), a);
#pragma unroll
        for (int n = 0; n < 4; ++n) gl_mma(acc[m][n], a, b[n >> 1][(n & 1) * 2], b[n >> 1][(n & 1) * 2 + 1]);
      }
    }
    __syncwarp();                  // every lane is done with the stage
    issue(i + 2);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncwarp();
  // park the warp's sums in its own buffers
  float* sum = reinterpret_cast<float*>(buf);
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int r = m * 16 + (lane >> 2), f = n * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(sum + r * GL_SUM_LD + f) = make_float2(acc[m][n][0], acc[m][n][1]);
      *reinterpret_cast<float2*>(sum + (r + 8) * GL_SUM_LD + f) = make_float2(acc[m][n][2], acc[m][n][3]);
    }
  __syncthreads();
  // over the warps, into the first warp's place (a thread reads and writes the same elements)
  const float* all = reinterpret_cast<const float*>(gl_smem);
  float* cta_sum = reinterpret_cast<float*>(gl_smem);
  for (int e = tid; e < GL_ROWS * GL_F; e += GL_THREADS) {
    const int at = (e / GL_F) * GL_SUM_LD + e % GL_F;
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < GL_WARPS; ++w) v += all[(size_t)w * (warp_bytes / 4) + at];
    cta_sum[at] = v;
  }
  if (n_cta > 1) cluster.sync();
  else __syncthreads();
  // over the CTAs of the cluster: rows rank, rank + n_cta, ...
  for (int e = tid; e < (GL_ROWS / n_cta) * GL_F; e += GL_THREADS) {
    const int r = (e / GL_F) * n_cta + rank, f = e % GL_F;
    float v = 0.f;
    for (int c = 0; c < n_cta; ++c) {
      const float* s = n_cta > 1 ? cluster.map_shared_rank(cta_sum, c) : cta_sum;
      v += s[r * GL_SUM_LD + f];
    }
    if (r < rows && f0 + f < p.F) {
      const size_t idx = (size_t)(t0 + r) * p.out_ld + f0 + f;
      if (p.out_f32) ((float*)p.out)[idx] = p.residual ? v + ((const float*)p.residual)[idx] : v;
      else ((__nv_bfloat16*)p.out)[idx] = __float2bfloat16(p.residual ? v + __bfloat162float(((const __nv_bfloat16*)p.residual)[idx]) : v);
    }
  }
  if (n_cta > 1) cluster.sync();   // nobody leaves while its sums are read
}

}  // namespace skein

// K a multiple of 8, rows of x and w on 16-byte boundaries. Returns -1 for shapes it does not take.
extern "C" int skein_gemm_small(const void* x, long long x_ld, const void* w, void* out, long long out_ld, const void* residual, int T, int F, int K,
                                int out_f32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (T < 1 || F < 1 || K < 8 || K % 8 != 0 || x_ld % 8 != 0 || (uintptr_t)x % 16 != 0 || (uintptr_t)w % 16 != 0) return -1;
  static bool attr_set[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -4;
  if (!attr_set[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(gemm_small_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, GL_SMEM);
    if (e != cudaSuccess) return (int)e;
    attr_set[dev] = true;
  }
  const int ft = (F + GL_F - 1) / GL_F, rt = (T + GL_ROWS - 1) / GL_ROWS, pieces = (K + GL_K - 1) / GL_K;
  int cluster = 1;                 // more CTAs while the pieces feed their warps and the GPU has room
  while (cluster < GL_MAX_CLUSTER && cluster * GL_WARPS < pieces && 2ll * cluster * ft * rt <= 148) cluster *= 2;
  const int stages = pieces > cluster * GL_WARPS ? 2 : 1;
  const GemmSmallParams p{(const __nv_bfloat16*)x, (const __nv_bfloat16*)w, out, residual, x_ld, out_ld, T, F, K, out_f32, stages};
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(cluster, ft, rt);
  cfg.blockDim = dim3(GL_THREADS);
  cfg.dynamicSmemBytes = (size_t)GL_WARPS * stages * GL_STAGE;
  cfg.stream = (cudaStream_t)stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cluster;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  return (int)cudaLaunchKernelEx(&cfg, gemm_small_kernel, p);
}
