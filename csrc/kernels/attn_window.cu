// Sliding-window attention with a norm over the whole query and key projections: the kernel in front of it, and a plain
// attention kernel for every head size and for fp32.
//
//   window_append     per token: q and k divided by the root mean square of all their rows at once, times a weight, the first
//                     rot_dims dimensions of every head rotated (pairs i, i + rot_dims / 2); q back in place, k and v into the
//                     paged cache
//   window_attn_rows  attention of single rows: position i sees the keys j with 0 <= i - j < window
//
// Cache page: [kv_heads, page_size, dim] keys, then [kv_heads, page_size, vdim] values (with dim == vdim the layout of the
// other attention kernels, [2, kv_heads, page_size, dim]). cos/sin: fp32 table [max_pos, rot_dims / 2, 2] made on the host.
// Compiled without fast-math.
#include "ptx.cuh"
#include "launch.cuh"
#include "vec.cuh"
#include <math.h>

namespace skein {

struct WindowAppendParams {
  void* q;                   // [T, ld] activation type, heads * dim columns; rotated in place
  const void* k;             // [T, ld] kv_heads * dim columns
  const void* v;             // [T, ld] kv_heads * vdim columns
  const float* q_norm;       // [heads * dim]
  const float* k_norm;       // [kv_heads * dim]
  const float* cos_sin;      // [max_pos, rot_dims / 2, 2]
  const int* positions;      // [T], -1: padding row
  const int* seq_of_token;   // [T] row of block_table, or null (row = token)
  const int* block_table;    // [S, max_blocks]
  void* cache;               // [pages, kv_heads * page_size * (dim + vdim)]
  int* status;
  long long ld;
  int H, K, D, V, rot, max_pos, max_blocks, num_pages, page_size;
  float eps;
};

__device__ __forceinline__ float wa_block_sum(float v, float* sh) {
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t += sh[i];
  __syncthreads();
  return t;
}

// grid (T, 2): queries, then keys and values. VEC elements per access; a rotated pair is two accesses rot / 2 apart.
template <typename T, int VEC>
__global__ void __launch_bounds__(1024) window_append_kernel(const WindowAppendParams p) {
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, pos = p.positions[t];
  if (pos < 0) return;
  if (pos >= p.max_pos) { if (threadIdx.x == 0) report_status(p.status, ST_BAD_INDEX, pos); return; }
  const bool keys = blockIdx.y == 1;
  const int heads = keys ? p.K : p.H, n = heads * p.D, half = p.rot / 2;
  const T* src = (keys ? (const T*)p.k : (const T*)p.q) + (size_t)t * p.ld;
  const float* nw = keys ? p.k_norm : p.q_norm;
  T *kd = nullptr, *vd = nullptr;
  if (keys) {
    const int seq = p.seq_of_token ? p.seq_of_token[t] : t;
    const int page = p.block_table[(size_t)seq * p.max_blocks + pos / p.page_size];
    if (page < 0 || page >= p.num_pages) { if (threadIdx.x == 0) report_status(p.status, ST_BAD_INDEX, page); return; }
    kd = (T*)p.cache + (size_t)page * p.K * p.page_size * (p.D + p.V) + (size_t)(pos % p.page_size) * p.D;
    vd = (T*)p.cache + (size_t)page * p.K * p.page_size * (p.D + p.V) + (size_t)p.K * p.page_size * p.D + (size_t)(pos % p.page_size) * p.V;
  }
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < n; i += blockDim.x * VEC) {
    float a[VEC];
    load_v<T, VEC>(src + i, a);
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss += a[k] * a[k];
  }
  const float r = 1.f / sqrtf(wa_block_sum(ss, sh) / (float)n + p.eps);
  const float2* cs = reinterpret_cast<const float2*>(p.cos_sin) + (size_t)pos * half;
  // an element of the first half of the rotated part takes its partner along; the partner's own turn is skipped
  for (int i = threadIdx.x * VEC; i < n; i += blockDim.x * VEC) {
    const int h = i / p.D, d = i % p.D;
    if (d >= half && d < p.rot) continue;
    float a[VEC], w[VEC];
    load_v<T, VEC>(src + i, a);
    load_v<float, VEC>(nw + i, w);
#pragma unroll
    for (int k = 0; k < VEC; ++k) a[k] *= r * w[k];
    T* dst = keys ? kd + (size_t)h * p.page_size * p.D + d : (T*)p.q + (size_t)t * p.ld + i;
    if (d < half) {
      float b[VEC];
      load_v<T, VEC>(src + i + half, b);
      load_v<float, VEC>(nw + i + half, w);
#pragma unroll
      for (int k = 0; k < VEC; ++k) {
        const float2 c = cs[d + k];
        const float y = b[k] * r * w[k];
        b[k] = y * c.x + a[k] * c.y;
        a[k] = a[k] * c.x - y * c.y;
      }
      store_v<T, VEC>(dst + half, b);
    }
    store_v<T, VEC>(dst, a);
  }
  if (!keys) return;
  const T* vs = (const T*)p.v + (size_t)t * p.ld;
  for (int i = threadIdx.x; i < p.K * p.V; i += blockDim.x) vd[(size_t)(i / p.V) * p.page_size * p.V + i % p.V] = vs[i];
}

struct WindowAttnParams {
  const void* q;             // [T, ld] rotated queries
  const void* cache;
  const int* positions;
  const int* seq_of_token;
  const int* block_table;
  void* out;                 // [T, out_ld] heads * vdim columns
  int* status;
  long long ld, out_ld;
  int H, K, D, V, max_blocks, num_pages, page_size, window;
  float scale, out_scale;
};

constexpr int WR_TILE = 128;       // keys per round, one per thread

// grid (T, H), 128 threads. Scores of a tile of keys, running softmax, then every thread sums the values of its output columns.
template <typename T>
__global__ void __launch_bounds__(WR_TILE) window_attn_rows_kernel(const WindowAttnParams p) {
  extern __shared__ float q_s[];           // [D] query, then [V] sums
  __shared__ float prob[WR_TILE];
  __shared__ const T* page_s[WR_TILE];
  __shared__ float red[4];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, pos = p.positions[t];
  if (pos < 0) return;
  const int kvh = h / (p.H / p.K), seq = p.seq_of_token ? p.seq_of_token[t] : t;
  float* o_s = q_s + p.D;
  const T* q = (const T*)p.q + (size_t)t * p.ld + (size_t)h * p.D;
  for (int i = tid; i < p.D; i += WR_TILE) q_s[i] = to_f<T>(q[i]);
  for (int i = tid; i < p.V; i += WR_TILE) o_s[i] = 0.f;
  const int lo = p.window > 0 && pos - p.window + 1 > 0 ? pos - p.window + 1 : 0;
  const size_t page_elems = (size_t)p.K * p.page_size * (p.D + p.V);
  float m = -INFINITY, l = 0.f;
  for (int j0 = lo; j0 <= pos; j0 += WR_TILE) {
    __syncthreads();
    const int j = j0 + tid, cnt = min(WR_TILE, pos + 1 - j0);
    float s = -INFINITY;
    if (j <= pos) {
      int page = p.block_table[(size_t)seq * p.max_blocks + j / p.page_size];
      if (page < 0 || page >= p.num_pages) { report_status(p.status, ST_BAD_INDEX, page); page = 0; }
      const T* base = (const T*)p.cache + (size_t)page * page_elems;
      const T* k = base + ((size_t)kvh * p.page_size + j % p.page_size) * p.D;
      page_s[tid] = base + (size_t)p.K * p.page_size * p.D + ((size_t)kvh * p.page_size + j % p.page_size) * p.V;
      float a = 0.f;
      for (int d = 0; d < p.D; ++d) a = fmaf(q_s[d], to_f<T>(k[d]), a);
      s = a * p.scale;
    }
    float mx = s;
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    if ((tid & 31) == 0) red[tid >> 5] = mx;
    __syncthreads();
    const float mn = fmaxf(m, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
    const float keep = m == -INFINITY ? 0.f : expf(m - mn), e = j <= pos ? expf(s - mn) : 0.f;
    m = mn;
    prob[tid] = e;
    float sum = e;
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    __syncthreads();
    if ((tid & 31) == 0) red[tid >> 5] = sum;
    __syncthreads();
    l = l * keep + red[0] + red[1] + red[2] + red[3];
    for (int d = tid; d < p.V; d += WR_TILE) {
      float a = o_s[d] * keep;
      for (int i = 0; i < cnt; ++i) a = fmaf(prob[i], to_f<T>(page_s[i][d]), a);
      o_s[d] = a;
    }
  }
  T* out = (T*)p.out + (size_t)t * p.out_ld + (size_t)h * p.V;
  for (int d = tid; d < p.V; d += WR_TILE) out[d] = from_f<T>(o_s[d] / l * p.out_scale);
}

}  // namespace skein

extern "C" int skein_window_append(void* q, const void* k, const void* v, long long ld, const float* q_norm, const float* k_norm, const float* cos_sin,
                                   const int* positions, const int* seq_of_token, const int* block_table, void* cache, int* status, int T, int H, int K,
                                   int D, int V, int rot, int max_pos, int max_blocks, int num_pages, int page_size, float eps, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (rot % 2 != 0 || rot > D) return -1;
  WindowAppendParams p{q, k, v, q_norm, k_norm, cos_sin, positions, seq_of_token, block_table, cache, status, ld, H, K, D, V, rot, max_pos, max_blocks,
                       num_pages, page_size, eps};
  const bool v4 = D % 4 == 0 && (rot / 2) % 4 == 0 && ld % 4 == 0 && (size_t)K * page_size * (D + V) % 4 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)k % 16 == 0;
  const dim3 grid(T, 2);
  int th = 256;                     // few rows: up to one access per thread
  while (T <= 512 && th < 1024 && th * (v4 ? 4 : 1) < H * D) th *= 2;
  const dim3 b(th);
  cudaStream_t s = (cudaStream_t)stream;
  if (fp32) return (int)(v4 ? launch_pdl(window_append_kernel<float, 4>, grid, b, 0, s, p) : launch_pdl(window_append_kernel<float, 1>, grid, b, 0, s, p));
  return (int)(v4 ? launch_pdl(window_append_kernel<__nv_bfloat16, 4>, grid, b, 0, s, p)
                  : launch_pdl(window_append_kernel<__nv_bfloat16, 1>, grid, b, 0, s, p));
}

extern "C" int skein_window_attn_rows(const void* q, long long ld, const void* cache, const int* positions, const int* seq_of_token,
                                      const int* block_table, void* out, long long out_ld, int* status, int T, int H, int K, int D, int V, int max_blocks,
                                      int num_pages, int page_size, int window, float scale, float out_scale, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (H % K != 0 || (D + V) * 4 > 40 * 1024) return -1;
  WindowAttnParams p{q, cache, positions, seq_of_token, block_table, out, status, ld, out_ld, H, K, D, V, max_blocks, num_pages, page_size, window, scale,
                     out_scale};
  const dim3 grid(T, H);
  const size_t sm = (size_t)(D + V) * 4;
  cudaStream_t s = (cudaStream_t)stream;
  return (int)(fp32 ? launch_pdl(window_attn_rows_kernel<float>, grid, dim3(WR_TILE), sm, s, p)
                    : launch_pdl(window_attn_rows_kernel<__nv_bfloat16>, grid, dim3(WR_TILE), sm, s, p));
}
