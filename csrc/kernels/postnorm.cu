// Kernels of post-norm blocks whose residual stream is fp32: embedding, the short causal convolution in front of a mixer,
// residual sum + RMS norm with one gain for all coordinates (alone, with the next block's convolution, or with the MoE
// router and expert-sorted scatter), the polynomial activation.
//
//   conv_input       h_t = x_t + sum_j w[j] * x_(t - taps + 1 + j)         (per channel, zeros before position 0)
//   post_norm        x <- g * v / sqrt(mean(v^2) + eps),  v = alpha * x + y,   y a row or a weighted sum of expert rows
//   poly_norm        a N(z) + b N(z^2) + c N(z^3) + e,   N(v) = v / sqrt(mean(v^2) + eps)
//
// The convolution's last inputs are part of a sequence's cache and live with its pages: every page has R = min(taps, page
// size) tail rows, position p's input sits in row (p mod page size) mod R of p's page (taps - 1 rows would hold the state; with
// one more, a decode step never overwrites a row it reads and can be run again). So a page of the prefix cache
// brings the convolution's state along, freeing a sequence frees it, and a batch row needs no state slot of its own. The
// values kept are in the activation type; the convolution reads the same rounded values inside a chunk, so that a result does
// not depend on how a prompt was cut.
//
// T is the activation type (bf16, or fp32 when a model runs in 32-bit); residual stream, norms and sums are fp32 always.
#include "ptx.cuh"
#include "launch.cuh"
#include "route.cuh"
#include "vec.cuh"
#include <cuda_bf16.h>
#include <math.h>

namespace skein {

constexpr int PN_MAX_TAPS = 32;

__device__ __forceinline__ float pn_block_sum(float v, float* sh) {
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (l == 0) sh[w] = v;
  __syncthreads();
  float t = (l < nw) ? sh[l] : 0.f;
  for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
  __syncthreads();
  return t;
}

// ---- convolution state ----------------------------------------------------------------------------
struct ConvParams {
  const float* w;            // [taps, C]
  void* tail;                // [pages, R, C] activation type
  const int* positions;      // [T]
  const int* seq_of_token;   // [T] row of block_table, or null (row = token)
  const int* q_start;        // [S] first row of each sequence's chunk, or null (every row is its own chunk)
  const int* block_table;    // [S, max_blocks]
  int* status;
  int max_blocks, num_pages, page_size, R, taps, C;
};

// Where the tap j steps back (j = 1 .. taps - 1) of row t finds its input: a row of x inside the chunk (in_chunk[j] >= 0), a
// tail row of the cache, or nothing (before the start).
template <typename T>
__device__ __forceinline__ const T* conv_tail_row(const ConvParams& c, int seq, int q) {
  const int page = c.block_table[(size_t)seq * c.max_blocks + q / c.page_size];
  if (page < 0 || page >= c.num_pages) { report_status(c.status, ST_BAD_INDEX, page); return nullptr; }
  return reinterpret_cast<const T*>(c.tail) + ((size_t)page * c.R + (q % c.page_size) % c.R) * c.C;
}

// one CTA per row
template <typename T, int V>
__global__ void __launch_bounds__(256) conv_input_kernel(const float* __restrict__ x, T* __restrict__ h, const ConvParams c, int write_tail) {
  __shared__ const T* tail_s[PN_MAX_TAPS];
  __shared__ int row_s[PN_MAX_TAPS];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int pos = c.positions[t];
  const int seq = c.seq_of_token ? c.seq_of_token[t] : t;
  const int first = c.q_start ? c.q_start[seq] : t;
  if ((int)threadIdx.x < c.taps && threadIdx.x > 0) {
    const int j = threadIdx.x, q = pos - j;
    row_s[j] = (q >= 0 && t - j >= first) ? t - j : -1;
    tail_s[j] = (q >= 0 && t - j < first) ? conv_tail_row<T>(c, seq, q) : nullptr;
  }
  if (threadIdx.x == 0) tail_s[0] = (write_tail && pos >= 0 && c.R > 0) ? conv_tail_row<T>(c, seq, pos) : nullptr;
  __syncthreads();
  for (int i = threadIdx.x * V; i < c.C; i += blockDim.x * V) {
    float xv[V], acc[V], w[V], v[V];
    load_v<float, V>(x + (size_t)t * c.C + i, xv);
    load_v<float, V>(c.w + (size_t)(c.taps - 1) * c.C + i, w);
#pragma unroll
    for (int k = 0; k < V; ++k) acc[k] = w[k] * to_f<T>(from_f<T>(xv[k]));
    for (int j = 1; j < c.taps; ++j) {
      if (row_s[j] >= 0) {
        load_v<float, V>(x + (size_t)row_s[j] * c.C + i, v);
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = to_f<T>(from_f<T>(v[k]));
      } else if (tail_s[j] != nullptr) {
        load_v<T, V>(tail_s[j] + i, v);
      } else {
        continue;
      }
      load_v<float, V>(c.w + (size_t)(c.taps - 1 - j) * c.C + i, w);
#pragma unroll
      for (int k = 0; k < V; ++k) acc[k] += w[k] * v[k];
    }
    if (tail_s[0] != nullptr) store_v<T, V>(const_cast<T*>(tail_s[0]) + i, xv);
#pragma unroll
    for (int k = 0; k < V; ++k) acc[k] += xv[k];
    store_v<T, V>(h + (size_t)t * c.C + i, acc);
  }
}

// ---- residual sum + norm ---------------------------------------------------------------------------
struct PostNormParams {
  const float* x;            // [B, C] residual stream
  const void* y;             // [rows, C] activation type, or null
  const int* row_idx;        // [B, topk] rows of y, or null (row = b)
  const float* row_w;        // [B, topk] weights, or null
  const float* gain;         // [1]
  const float* final_gain;   // [1] or null: act_out is the norm of the NEW residual with this gain (before the output projection)
  float* x_out;              // [B, C]
  void* act_out;             // [B, C] activation type: the new residual (or its convolution / final norm), or null
  int* status;
  float alpha, eps;
  int C, topk;
};

// v = alpha * x + y of V elements at column i
template <typename T, int V>
__device__ __forceinline__ void post_sum(const PostNormParams& p, int b, int i, float* a) {
  load_v<float, V>(p.x + (size_t)b * p.C + i, a);
#pragma unroll
  for (int k = 0; k < V; ++k) a[k] *= p.alpha;
  if (p.y == nullptr) return;
  const T* y = (const T*)p.y;
  const int nk = p.row_idx ? p.topk : 1;
  for (int j0 = 0; j0 < nk; j0 += 8) {       // rows in batches of 8: all loads of a batch are issued before the first is used
    float v[8][V], w8[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      w8[j] = 0.f;
      if (j0 + j < nk) {
        const int row = p.row_idx ? p.row_idx[(size_t)b * p.topk + j0 + j] : b;
        w8[j] = row < 0 ? 0.f : (p.row_w ? p.row_w[(size_t)b * p.topk + j0 + j] : 1.f);
        load_v<T, V>(y + (size_t)(row < 0 ? 0 : row) * p.C + i, v[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (j0 + j < nk)
#pragma unroll
        for (int k = 0; k < V; ++k) a[k] += w8[j] * v[j][k];
  }
}

// One CTA per row; the row's sums are parked in dynamic shared memory (C floats) between the two passes. CONV: act_out is
// the input of the next block's mixer, x + convolution (decode: every row is its own sequence, its last inputs come from the
// cache, and the row's own input is appended there).
template <typename T, int V, bool CONV>
__global__ void __launch_bounds__(512) post_norm_kernel(const PostNormParams p, const ConvParams c) {
  extern __shared__ __align__(16) float row_sm[];
  __shared__ float sh[32];
  __shared__ const T* tail_s[PN_MAX_TAPS];
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x;
  if (CONV) {
    const int pos = c.positions[b];
    if ((int)threadIdx.x < c.taps) {
      const int j = threadIdx.x, q = pos - j;
      tail_s[j] = (q >= 0 && pos >= 0 && c.R > 0) ? conv_tail_row<T>(c, b, q) : nullptr;
    }
  }
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < p.C; i += blockDim.x * V) {
    float a[V];
    post_sum<T, V>(p, b, i, a);
#pragma unroll
    for (int k = 0; k < V; ++k) { row_sm[i + k] = a[k]; ss += a[k] * a[k]; }
  }
  const float tot = pn_block_sum(ss, sh);     // (also the barrier behind tail_s)
  const float scale = p.gain[0] / sqrtf(tot / (float)p.C + p.eps);
  float scale2 = 1.f;
  if (p.final_gain != nullptr) {
    // mean square of the new residual follows from the old one's: every element is multiplied by `scale`
    scale2 = p.final_gain[0] / sqrtf(tot * scale * scale / (float)p.C + p.eps);
  }
  for (int i = threadIdx.x * V; i < p.C; i += blockDim.x * V) {
    float xv[V];
#pragma unroll
    for (int k = 0; k < V; ++k) xv[k] = row_sm[i + k] * scale;
    if (p.x_out) store_v<float, V>(p.x_out + (size_t)b * p.C + i, xv);
    if (CONV) {
      float acc[V], w[V], v[V];
      load_v<float, V>(c.w + (size_t)(c.taps - 1) * c.C + i, w);
#pragma unroll
      for (int k = 0; k < V; ++k) acc[k] = w[k] * to_f<T>(from_f<T>(xv[k]));
      for (int j = 1; j < c.taps; ++j) {
        if (tail_s[j] == nullptr) continue;
        load_v<T, V>(tail_s[j] + i, v);
        load_v<float, V>(c.w + (size_t)(c.taps - 1 - j) * c.C + i, w);
#pragma unroll
        for (int k = 0; k < V; ++k) acc[k] += w[k] * v[k];
      }
      if (tail_s[0] != nullptr) store_v<T, V>(const_cast<T*>(tail_s[0]) + i, xv);
#pragma unroll
      for (int k = 0; k < V; ++k) xv[k] += acc[k];
    } else if (p.final_gain != nullptr) {
#pragma unroll
      for (int k = 0; k < V; ++k) xv[k] *= scale2;
    }
    if (p.act_out) store_v<T, V>((T*)p.act_out + (size_t)b * p.C + i, xv);
  }
}

// The same for a bf16 model's decode step, followed in the same launch by the router and the scatter of the row into
// expert-sorted order (route.cuh). One CTA per row, all resident at once; a thread owns 8 consecutive elements per pass.
template <int MAX_PASSES>
__global__ void __launch_bounds__(512) post_norm_route_kernel(const PostNormParams p, const RouteParams r, const SkeinRouteRule rule) {
  __shared__ float sh[32];
  __shared__ RouteShared rs;
  __shared__ int sel_id[NR_MAX_K];
  __shared__ float sel_w[NR_MAX_K];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, T = gridDim.x;
  const int per_pass = blockDim.x * 8;
  float vals[MAX_PASSES][8];
  float ss = 0.f;
#pragma unroll
  for (int ps = 0; ps < MAX_PASSES; ++ps) {
    const int h = ps * per_pass + tid * 8;
    if (h >= p.C) break;
    post_sum<__nv_bfloat16, 4>(p, t, h, vals[ps]);
    post_sum<__nv_bfloat16, 4>(p, t, h + 4, vals[ps] + 4);
#pragma unroll
    for (int k = 0; k < 8; ++k) ss += vals[ps][k] * vals[ps][k];
  }
  const float tot = pn_block_sum(ss, sh);
  const float scale = p.gain[0] / sqrtf(tot / (float)p.C + p.eps);
  uint4 nb[MAX_PASSES];
#pragma unroll
  for (int ps = 0; ps < MAX_PASSES; ++ps) {
    const int h = ps * per_pass + tid * 8;
    if (h >= p.C) break;
#pragma unroll
    for (int k = 0; k < 8; ++k) vals[ps][k] *= scale;
    float* xo = p.x_out + (size_t)t * p.C + h;
    store_v<float, 4>(xo, vals[ps]);
    store_v<float, 4>(xo + 4, vals[ps] + 4);
    __nv_bfloat162* ob = reinterpret_cast<__nv_bfloat162*>(&nb[ps]);
#pragma unroll
    for (int k = 0; k < 4; ++k) ob[k] = __floats2bfloat162_rn(vals[ps][2 * k], vals[ps][2 * k + 1]);
  }
  route_partial_logits<MAX_PASSES>(nb, true, r.wg, r.E, p.C, rs);
  __syncthreads();
  for (int e = tid; e < r.E; e += blockDim.x) rs.logit[e] = route_sum_logit(rs, e);
  __syncthreads();
  if (tid < 32) {
    select_grouped_warp<NR_MAX_E>(rs.logit, r.E, r.topk, rule, sel_id, sel_w);
    if (tid == 0) {
      for (int j = 0; j < r.topk; ++j) {
        r.expert_ids[t * r.topk + j] = sel_id[j];
        r.expert_w[t * r.topk + j] = sel_w[j];
      }
      route_publish_and_wait(r, p.status, t, T, rs);
    }
  }
  __syncthreads();
  if (!rs.barrier_ok) return;   // the counters stay dirty: the host clears them when it handles the status
  route_scatter<MAX_PASSES>(r, nb, true, p.C, t, T, rs);
}

// ---- polynomial activation ----------------------------------------------------------------------------
// one CTA per row of F values, parked in dynamic shared memory
template <typename T, int V>
__global__ void __launch_bounds__(1024) poly_norm_kernel(const T* __restrict__ z, const float* __restrict__ act, T* __restrict__ out, int F, float eps) {
  extern __shared__ __align__(16) float row_sm[];
  __shared__ float sh[3][32];
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x;
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll 4
  for (int i = threadIdx.x * V; i < F; i += blockDim.x * V) {
    float v[V];
    load_v<T, V>(z + (size_t)b * F + i, v);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      row_sm[i + k] = v[k];
      const float q = v[k] * v[k];
      s1 += q; s2 += q * q; s3 += q * q * q;
    }
  }
  for (int o = 16; o > 0; o >>= 1) {
    s1 += __shfl_xor_sync(0xffffffffu, s1, o);
    s2 += __shfl_xor_sync(0xffffffffu, s2, o);
    s3 += __shfl_xor_sync(0xffffffffu, s3, o);
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) { sh[0][warp] = s1; sh[1][warp] = s2; sh[2][warp] = s3; }
  __syncthreads();
  s1 = lane < nw ? sh[0][lane] : 0.f; s2 = lane < nw ? sh[1][lane] : 0.f; s3 = lane < nw ? sh[2][lane] : 0.f;
  for (int o = 16; o > 0; o >>= 1) {
    s1 += __shfl_xor_sync(0xffffffffu, s1, o);
    s2 += __shfl_xor_sync(0xffffffffu, s2, o);
    s3 += __shfl_xor_sync(0xffffffffu, s3, o);
  }
  const float n = (float)F;
  const float ca = act[0] / sqrtf(s1 / n + eps), cb = act[1] / sqrtf(s2 / n + eps), cc = act[2] / sqrtf(s3 / n + eps), ce = act[3];
  for (int i = threadIdx.x * V; i < F; i += blockDim.x * V) {
    float o[V];
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const float v = row_sm[i + k];
      o[k] = ((cc * v + cb) * v + ca) * v + ce;
    }
    store_v<T, V>(out + (size_t)b * F + i, o);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256) embed_f32_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out, int C, int rows) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, id = ids[t];
  const bool ok = id >= 0 && id < rows;
  for (int i = threadIdx.x * V; i < C; i += blockDim.x * V) {
    float v[V];
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] = 0.f;
    if (ok) load_v<T, V>(table + (size_t)id * C + i, v);
    store_v<float, V>(out + (size_t)t * C + i, v);
  }
}

static int row_threads(int n, int v, int cap) {
  int th = (n / v + 31) / 32 * 32;
  if (th < 32) th = 32;
  return th > cap ? cap : th;
}
constexpr int PN_MAX_ROW = 48 * 1024 / 4 - 512;   // floats of a row that fit the default dynamic shared memory beside the static part

// rows longer than the default 48 KB of dynamic shared memory need the kernel's limit raised once
template <typename F>
static cudaError_t allow_smem(F fn, int bytes) {
  return bytes > PN_MAX_ROW * 4 ? cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes) : cudaSuccess;
}

}  // namespace skein

extern "C" int skein_embed_f32(const int* ids, const void* table, float* out, int T, int C, int rows, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = C % 4 == 0;
  const dim3 b(row_threads(C, v4 ? 4 : 1, 256));
  if (fp32) return (int)(v4 ? launch_pdl(embed_f32_kernel<float, 4>, dim3(T), b, 0, s, ids, (const float*)table, out, C, rows)
                            : launch_pdl(embed_f32_kernel<float, 1>, dim3(T), b, 0, s, ids, (const float*)table, out, C, rows));
  return (int)(v4 ? launch_pdl(embed_f32_kernel<__nv_bfloat16, 4>, dim3(T), b, 0, s, ids, (const __nv_bfloat16*)table, out, C, rows)
                  : launch_pdl(embed_f32_kernel<__nv_bfloat16, 1>, dim3(T), b, 0, s, ids, (const __nv_bfloat16*)table, out, C, rows));
}

// taps up to 32. seq_of_token / q_start null: decode rows (each its own sequence). write_tail appends each row's input to the
// cache (decode rows only: rows of one chunk read their predecessors' inputs, which are appended afterwards, see latent.cu).
extern "C" int skein_conv_input(const float* x, void* h, const float* w, void* tail, const int* positions, const int* seq_of_token,
                                const int* q_start, const int* block_table, int* status, int T, int C, int taps, int R, int page_size,
                                int max_blocks, int num_pages, int write_tail, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (taps < 1 || taps > PN_MAX_TAPS || (taps > 1 && R < 1)) return -1;
  ConvParams c{w, tail, positions, seq_of_token, q_start, block_table, status, max_blocks, num_pages, page_size, R, taps, C};
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = C % 4 == 0;
  const dim3 b(row_threads(C, v4 ? 4 : 1, 256));
  if (fp32) return (int)(v4 ? launch_pdl(conv_input_kernel<float, 4>, dim3(T), b, 0, s, x, (float*)h, c, write_tail)
                            : launch_pdl(conv_input_kernel<float, 1>, dim3(T), b, 0, s, x, (float*)h, c, write_tail));
  return (int)(v4 ? launch_pdl(conv_input_kernel<__nv_bfloat16, 4>, dim3(T), b, 0, s, x, (__nv_bfloat16*)h, c, write_tail)
                  : launch_pdl(conv_input_kernel<__nv_bfloat16, 1>, dim3(T), b, 0, s, x, (__nv_bfloat16*)h, c, write_tail));
}

// conv_w null: no convolution. final_gain null: act_out holds the new residual.
extern "C" int skein_post_norm(const float* x, const void* y, const int* row_idx, const float* row_w, const float* gain,
                               const float* final_gain, float* x_out, void* act_out, float alpha, float eps, int B, int C, int topk,
                               const float* conv_w, void* tail, const int* positions, const int* block_table, int* status, int taps, int R,
                               int page_size, int max_blocks, int num_pages, int fp32, void* stream) {
  using namespace skein;
  if (B == 0) return 0;
  if (C < 1 || C * 4 > 200 * 1024) return -1;
  if (conv_w != nullptr && (taps < 1 || taps > PN_MAX_TAPS || (taps > 1 && R < 1))) return -1;
  PostNormParams p{x, y, row_idx, row_w, gain, final_gain, x_out, act_out, status, alpha, eps, C, topk};
  ConvParams c{conv_w, tail, positions, nullptr, nullptr, block_table, status, max_blocks, num_pages, page_size, R, taps, C};
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = C % 4 == 0;
  const dim3 b(row_threads(C, v4 ? 4 : 1, 512));
  const size_t sm = (size_t)C * 4;
  auto go = [&](auto fn) -> int {
    cudaError_t e = allow_smem(fn, (int)sm);
    return (int)(e != cudaSuccess ? e : launch_pdl(fn, dim3(B), b, sm, s, p, c));
  };
  const bool conv = conv_w != nullptr;
  if (fp32) return v4 ? (conv ? go(post_norm_kernel<float, 4, true>) : go(post_norm_kernel<float, 4, false>))
                      : (conv ? go(post_norm_kernel<float, 1, true>) : go(post_norm_kernel<float, 1, false>));
  return v4 ? (conv ? go(post_norm_kernel<__nv_bfloat16, 4, true>) : go(post_norm_kernel<__nv_bfloat16, 4, false>))
            : (conv ? go(post_norm_kernel<__nv_bfloat16, 1, true>) : go(post_norm_kernel<__nv_bfloat16, 1, false>));
}

// bf16, decode-sized batches: B at most `max_resident_ctas`, C a multiple of 8 up to 16384, E <= 64, topk <= 8.
extern "C" int skein_post_norm_route(const float* x, const void* y, const float* gain, float* x_out, float alpha, float eps, int B, int C,
                                     const void* wg, int E, int topk, int n_groups, int keep, int* expert_ids, float* expert_w, int* counts,
                                     int* offsets, int* row_of, int* src_token, void* xs, int* barrier, int max_resident_ctas, int* status,
                                     void* stream) {
  using namespace skein;
  if (B == 0) return 0;
  if (C % 8 != 0 || C > 4 * 512 * 8 || E > NR_MAX_E || topk > NR_MAX_K || topk > E || B * topk > NR_MAX_PAIRS) return -1;
  if (n_groups < 1 || n_groups > 64 || E % n_groups != 0 || keep < 1 || keep > n_groups || topk > keep * (E / n_groups)) return -1;
  if (B > max_resident_ctas) return -2;
  PostNormParams p{x, y, nullptr, nullptr, gain, nullptr, x_out, nullptr, status, alpha, eps, C, 0};
  RouteParams r;
  r.wg = (const __nv_bfloat16*)wg; r.expert_ids = expert_ids; r.expert_w = expert_w; r.counts = counts; r.offsets = offsets;
  r.row_of = row_of; r.src_token = src_token; r.xs = (__nv_bfloat16*)xs; r.barrier = barrier;
  r.E = E; r.topk = topk; r.e_first = 0; r.e_count = E;
  r.barrier_budget_ns = (unsigned long long)grid_barrier_budget_ms() * 1000000ull;
  int threads = row_threads(C, 8, 512);
  const int passes = (C + threads * 8 - 1) / (threads * 8);
  const SkeinRouteRule rule{n_groups, keep, ROUTE_SOFTMAX, 1, 0, 1.f};
  cudaStream_t s = (cudaStream_t)stream;
  if (passes <= 1) return (int)launch_pdl(post_norm_route_kernel<1>, dim3(B), dim3(threads), 0, s, p, r, rule);
  if (passes <= 2) return (int)launch_pdl(post_norm_route_kernel<2>, dim3(B), dim3(threads), 0, s, p, r, rule);
  return (int)launch_pdl(post_norm_route_kernel<4>, dim3(B), dim3(threads), 0, s, p, r, rule);
}

extern "C" int skein_poly_norm(const void* z, const float* act, void* out, int T, int F, float eps, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (F < 1 || F * 4 > 200 * 1024) return -1;
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = F % 4 == 0;
  const dim3 b(row_threads(F, v4 ? 4 : 1, T <= 256 ? 1024 : 256));     // few rows: more threads per row
  const size_t sm = (size_t)F * 4;
  auto go = [&](auto fn, auto zz, auto oo) -> int {
    cudaError_t e = allow_smem(fn, (int)sm);
    return (int)(e != cudaSuccess ? e : launch_pdl(fn, dim3(T), b, sm, s, zz, act, oo, F, eps));
  };
  if (fp32) return v4 ? go(poly_norm_kernel<float, 4>, (const float*)z, (float*)out) : go(poly_norm_kernel<float, 1>, (const float*)z, (float*)out);
  return v4 ? go(poly_norm_kernel<__nv_bfloat16, 4>, (const __nv_bfloat16*)z, (__nv_bfloat16*)out)
            : go(poly_norm_kernel<__nv_bfloat16, 1>, (const __nv_bfloat16*)z, (__nv_bfloat16*)out);
}
