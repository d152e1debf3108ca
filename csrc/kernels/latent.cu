// Latent attention (one cached row per token: a normed latent of kv_rank elements and one rotated key part shared by all
// heads): the small kernels around the projections, and a plain attention kernel for every size and for fp32.
//
//   latent_append   per token: norm the latent, rotate the key part, write the row to the paged cache (and, for a prefill
//                   chunk, to a dense copy that the expanded attention reads); norm the query latent; append the
//                   convolution's last inputs of the chunk (postnorm.cu)
//   rope_rows       rotate the query part of every head in place (prefill)
//   latent_gather   cached rows of the sequences -> one dense matrix
//   latent_attn     attention of single rows over the cache with the key expansion applied to the queries beforehand:
//                   score = (q_abs . c + rot(q_rot) . k_rot) * scale, output = sum_j p_j c_j per head
//
// Cache: [pages, page_size, kv_rank + rot_dim]. Rotation pairs neighbouring dimensions (2i, 2i + 1); cos/sin come from a
// host-built fp32 table [max_pos, rot/2, 2].
#include "ptx.cuh"
#include "launch.cuh"
#include <cuda_bf16.h>
#include <math.h>

namespace skein {

template <typename T> __device__ __forceinline__ float lt_f(T v);
template <> __device__ __forceinline__ float lt_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float lt_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T lt_t(float v);
template <> __device__ __forceinline__ float lt_t<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 lt_t<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

struct LatentAppendParams {
  const void* proj;          // [T, proj_ld]: query latent at column 0 (q_rank elements), cache row at column off_kv
  const float* q_norm;       // [q_rank] or null
  const float* kv_norm;      // [kv_rank]
  const float* cos_sin;      // [max_pos, rot/2, 2]
  const int* positions;      // [T], -1 = padding row
  const int* seq_of_token;   // [T] or null (row = token)
  const int* block_table;    // [S, max_blocks]
  void* cache;
  void* cq;                  // [T, q_rank] or null
  void* dense;               // [*, kv_rank + rot]: row dense_start[seq] + position, or null
  const int* dense_start;    // [S]
  const float* x;            // [T, C] inputs of the convolution, or null (decode rows append theirs in the norm kernel)
  void* tail;                // [pages, R, C]
  const int* seq_lens;       // [S] tokens after this chunk (with x)
  int* status;
  float eps;
  int proj_ld, off_kv, q_rank, kv_rank, rot, max_pos, max_blocks, num_pages, page_size, C, R, taps;
};

__device__ __forceinline__ float lt_block_sum(float v, float* sh) {
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (l == 0) sh[w] = v;
  __syncthreads();
  float t = (l < nw) ? sh[l] : 0.f;
  for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
  __syncthreads();
  return t;
}

// one CTA per token; a thread keeps up to LT_KEEP of its elements in registers between the sum and the store
constexpr int LT_THREADS = 256, LT_KEEP = 4;
template <typename T>
__global__ void __launch_bounds__(LT_THREADS) latent_append_kernel(const LatentAppendParams p) {
  __shared__ float sh[2][32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const T* row = (const T*)p.proj + (size_t)t * p.proj_ld;
  const T* ckr = row + p.off_kv;
  int pos = p.positions[t];
  const int seq = p.seq_of_token ? p.seq_of_token[t] : t;
  int page = -1;
  if (pos >= p.max_pos) { report_status(p.status, ST_BAD_INDEX, pos); pos = -1; }
  if (pos >= 0) {
    page = p.block_table[(size_t)seq * p.max_blocks + pos / p.page_size];
    if (page < 0 || page >= p.num_pages) { report_status(p.status, ST_BAD_INDEX, page); page = -1; }
  }
  float kv[LT_KEEP], sq = 0.f, sk = 0.f;
  for (int i = tid; i < p.q_rank; i += LT_THREADS) { const float v = lt_f<T>(row[i]); sq += v * v; }
#pragma unroll
  for (int k = 0; k < LT_KEEP; ++k) {
    const int i = tid + k * LT_THREADS;
    kv[k] = i < p.kv_rank ? lt_f<T>(ckr[i]) : 0.f;
    sk += kv[k] * kv[k];
  }
  for (int i = tid + LT_KEEP * LT_THREADS; i < p.kv_rank; i += LT_THREADS) { const float v = lt_f<T>(ckr[i]); sk += v * v; }
  for (int o = 16; o > 0; o >>= 1) { sq += __shfl_xor_sync(0xffffffffu, sq, o); sk += __shfl_xor_sync(0xffffffffu, sk, o); }
  if (lane == 0) { sh[0][warp] = sq; sh[1][warp] = sk; }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < LT_THREADS / 32; ++w) { sq += sh[0][w]; sk += sh[1][w]; }
  if (p.q_rank > 0) {
    const float inv = 1.f / sqrtf(sq / (float)p.q_rank + p.eps);
    T* cq = (T*)p.cq + (size_t)t * p.q_rank;
    for (int i = tid; i < p.q_rank; i += LT_THREADS) cq[i] = lt_t<T>(lt_f<T>(row[i]) * inv * p.q_norm[i]);
  }
  if (page < 0) return;      // padding row
  const int L = p.kv_rank + p.rot, slot = pos % p.page_size;
  const float inv = 1.f / sqrtf(sk / (float)p.kv_rank + p.eps);
  T* dst = (T*)p.cache + ((size_t)page * p.page_size + slot) * L;
  T* den = p.dense ? (T*)p.dense + (size_t)(p.dense_start[seq] + pos) * L : nullptr;
#pragma unroll
  for (int k = 0; k < LT_KEEP; ++k) {
    const int i = tid + k * LT_THREADS;
    if (i < p.kv_rank) {
      const T v = lt_t<T>(kv[k] * inv * p.kv_norm[i]);
      dst[i] = v;
      if (den) den[i] = v;
    }
  }
  for (int i = tid + LT_KEEP * LT_THREADS; i < p.kv_rank; i += LT_THREADS) {
    const T v = lt_t<T>(lt_f<T>(ckr[i]) * inv * p.kv_norm[i]);
    dst[i] = v;
    if (den) den[i] = v;
  }
  for (int i = tid; i < p.rot / 2; i += LT_THREADS) {
    const float2 cs = reinterpret_cast<const float2*>(p.cos_sin)[(size_t)pos * (p.rot / 2) + i];
    const float u = lt_f<T>(ckr[p.kv_rank + 2 * i]), w = lt_f<T>(ckr[p.kv_rank + 2 * i + 1]);
    const T a = lt_t<T>(u * cs.x - w * cs.y), b = lt_t<T>(w * cs.x + u * cs.y);
    dst[p.kv_rank + 2 * i] = a; dst[p.kv_rank + 2 * i + 1] = b;
    if (den) { den[p.kv_rank + 2 * i] = a; den[p.kv_rank + 2 * i + 1] = b; }
  }
  // the last taps - 1 inputs of the chunk, and of every page, are what later chunks (of this sequence, or of one that shares
  // the page) read
  if (p.x != nullptr && p.R > 0 && (pos >= p.seq_lens[seq] - (p.taps - 1) || slot >= p.page_size - (p.taps - 1))) {
    T* tl = (T*)p.tail + ((size_t)page * p.R + slot % p.R) * p.C;
    for (int i = tid; i < p.C; i += LT_THREADS) tl[i] = lt_t<T>(p.x[(size_t)t * p.C + i]);
  }
}

// q [T, ld]: head h's rotated part starts at column h * (D + rot) + D. grid = T.
template <typename T>
__global__ void __launch_bounds__(256) rope_rows_kernel(T* __restrict__ q, long long ld, const int* __restrict__ positions,
                                                        const float* __restrict__ cos_sin, int H, int D, int rot, int max_pos, int* status) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, pos = positions[t];
  if (pos < 0) return;
  if (pos >= max_pos) { report_status(status, ST_BAD_INDEX, pos); return; }
  const int half = rot / 2;
  for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
    const int h = i / half, k = i % half;
    T* r = q + (size_t)t * ld + (size_t)h * (D + rot) + D + 2 * k;
    const float2 cs = reinterpret_cast<const float2*>(cos_sin)[(size_t)pos * half + k];
    const float u = lt_f<T>(r[0]), w = lt_f<T>(r[1]);
    r[0] = lt_t<T>(u * cs.x - w * cs.y);
    r[1] = lt_t<T>(w * cs.x + u * cs.y);
  }
}

// grid = (blocks, sequences): rows [0, n) of every sequence's cache -> dense rows dense_start[s] + i, n = kv_len - q_len
template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const T* __restrict__ cache, const int* __restrict__ block_table, int max_blocks,
                                                            const int* __restrict__ kv_len, const int* __restrict__ q_len,
                                                            const int* __restrict__ dense_start, T* __restrict__ dense, int L, int page_size,
                                                            int num_pages, int* status) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.y, b = blockIdx.x;
  const int n = kv_len[s] - q_len[s];
  if (b * page_size >= n) return;
  const int page = block_table[(size_t)s * max_blocks + b];
  if (page < 0 || page >= num_pages) { if (threadIdx.x == 0) report_status(status, ST_BAD_INDEX, page); return; }
  int rows = n - b * page_size;
  if (rows > page_size) rows = page_size;
  const T* src = cache + (size_t)page * page_size * L;
  T* dst = dense + ((size_t)dense_start[s] + (size_t)b * page_size) * L;
  const long long bytes = (long long)rows * L * sizeof(T);
  if (((L * sizeof(T)) & 15) == 0) {
    for (long long i = threadIdx.x; i < bytes / 16; i += blockDim.x) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
  } else {
    for (long long i = threadIdx.x; i < (long long)rows * L; i += blockDim.x) dst[i] = src[i];
  }
}

// ---- plain attention of single rows -----------------------------------------------------------------------
struct LatentAttnParams {
  const void* q_abs;         // [T, H * kv_rank]
  const void* q;             // [T, q_ld] with head h's (unrotated) query part at column h * (D + rot) + D
  const float* cos_sin;
  const int* positions;      // [T]; row t sees positions 0 .. positions[t]; -1: padding row, output 0
  const int* seq_of_token;   // [T] or null
  const int* block_table;
  const void* cache;
  void* out;                 // [T, H * kv_rank]
  int* status;
  const float* sinks;        // [H] one more term exp(sinks[h]) in the denominator, or null
  long long q_ld;
  float scale;
  int H, D, rot, kv_rank, max_pos, max_blocks, num_pages, page_size;
};

constexpr int LA_THREADS = 128;

// grid = (T, H); dynamic shared memory: q [kv_rank + rot] + accumulator [kv_rank] + probabilities [128] (fp32) + page ids [128]
template <typename T>
__global__ void __launch_bounds__(LA_THREADS) latent_attn_rows_kernel(const LatentAttnParams p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int K = p.kv_rank, L = K + p.rot;
  float* qs = sm;
  float* acc = sm + L;
  float* pr = acc + K;
  const int pos = p.positions[t];
  T* out = (T*)p.out + (size_t)t * p.H * K + (size_t)h * K;
  if (pos < 0 || pos >= p.max_pos) {
    if (pos >= p.max_pos) report_status(p.status, ST_BAD_INDEX, pos);
    for (int i = tid; i < K; i += LA_THREADS) out[i] = lt_t<T>(0.f);
    return;
  }
  const int seq = p.seq_of_token ? p.seq_of_token[t] : t;
  const T* qa = (const T*)p.q_abs + (size_t)t * p.H * K + (size_t)h * K;
  const T* qr = (const T*)p.q + (size_t)t * p.q_ld + (size_t)h * (p.D + p.rot) + p.D;
  for (int i = tid; i < K; i += LA_THREADS) { qs[i] = lt_f<T>(qa[i]); acc[i] = 0.f; }
  for (int i = tid; i < p.rot / 2; i += LA_THREADS) {
    const float2 cs = reinterpret_cast<const float2*>(p.cos_sin)[(size_t)pos * (p.rot / 2) + i];
    const float u = lt_f<T>(qr[2 * i]), w = lt_f<T>(qr[2 * i + 1]);
    // rounded to the activation type, as a stored rotated query would be
    qs[K + 2 * i] = lt_f<T>(lt_t<T>(u * cs.x - w * cs.y));
    qs[K + 2 * i + 1] = lt_f<T>(lt_t<T>(w * cs.x + u * cs.y));
  }
  __syncthreads();
  const int n = pos + 1;
  float m = -INFINITY, l = 0.f;
  for (int j0 = 0; j0 < n; j0 += LA_THREADS) {
    const int j = j0 + tid;
    float s = -INFINITY;
    if (j < n) {
      int page = p.block_table[(size_t)seq * p.max_blocks + j / p.page_size];
      if (page < 0 || page >= p.num_pages) { report_status(p.status, ST_BAD_INDEX, page); page = 0; }
      const T* r = (const T*)p.cache + ((size_t)page * p.page_size + j % p.page_size) * L;
      float d = 0.f;
      for (int i = 0; i < L; ++i) d = fmaf(qs[i], lt_f<T>(r[i]), d);
      s = d * p.scale;
    }
    float mx = s;
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    if ((tid & 31) == 0) sh[tid >> 5] = mx;
    __syncthreads();
    mx = fmaxf(fmaxf(sh[0], sh[1]), fmaxf(sh[2], sh[3]));
    __syncthreads();
    const float mn = fmaxf(m, mx), al = m == -INFINITY ? 0.f : expf(m - mn);
    const float pj = j < n ? expf(s - mn) : 0.f;
    pr[tid] = pj;
    l = l * al + lt_block_sum(pj, sh);     // barriers inside: pr is visible behind it
    m = mn;
    const int cnt = min(LA_THREADS, n - j0);
    for (int i = tid; i < K; i += LA_THREADS) {
      float a = acc[i] * al;
      for (int jj = 0; jj < cnt; ++jj) {
        const int tk = j0 + jj;
        int page = p.block_table[(size_t)seq * p.max_blocks + tk / p.page_size];
        if (page < 0 || page >= p.num_pages) page = 0;
        a = fmaf(pr[jj], lt_f<T>(((const T*)p.cache)[((size_t)page * p.page_size + tk % p.page_size) * L + i]), a);
      }
      acc[i] = a;
    }
    __syncthreads();
  }
  float inv = 1.f / l;
  if (p.sinks) {
    const float sink = p.sinks[h], top = fmaxf(m, sink), e = expf(m - top);
    inv = e / (l * e + expf(sink - top));
  }
  for (int i = tid; i < K; i += LA_THREADS) out[i] = lt_t<T>(acc[i] * inv);
}

}  // namespace skein

extern "C" int skein_latent_append(const void* proj, int proj_ld, int off_kv, const float* q_norm, int q_rank, const float* kv_norm, int kv_rank,
                                   int rot, const float* cos_sin, int max_pos, const int* positions, const int* seq_of_token,
                                   const int* block_table, int max_blocks, void* cache, int num_pages, int page_size, void* cq, void* dense,
                                   const int* dense_start, const float* x, void* tail, const int* seq_lens, int C, int R, int taps, float eps,
                                   int T, int* status, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (rot % 2 != 0 || kv_rank < 1 || (q_rank > 0 && (q_norm == nullptr || cq == nullptr)) || (dense && !dense_start) || (x && !seq_lens)) return -1;
  LatentAppendParams p{proj, q_norm, kv_norm, cos_sin, positions, seq_of_token, block_table, cache, cq, dense, dense_start, x, tail, seq_lens,
                       status, eps, proj_ld, off_kv, q_rank, kv_rank, rot, max_pos, max_blocks, num_pages, page_size, C, R, taps};
  if (fp32) return (int)launch_pdl(latent_append_kernel<float>, dim3(T), dim3(LT_THREADS), 0, (cudaStream_t)stream, p);
  return (int)launch_pdl(latent_append_kernel<__nv_bfloat16>, dim3(T), dim3(LT_THREADS), 0, (cudaStream_t)stream, p);
}

extern "C" int skein_rope_rows(void* q, long long ld, const int* positions, const float* cos_sin, int T, int H, int D, int rot, int max_pos,
                               int* status, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (rot % 2 != 0) return -1;
  if (fp32) return (int)launch_pdl(rope_rows_kernel<float>, dim3(T), dim3(256), 0, (cudaStream_t)stream, (float*)q, ld, positions, cos_sin, H, D, rot, max_pos, status);
  return (int)launch_pdl(rope_rows_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, (cudaStream_t)stream, (__nv_bfloat16*)q, ld, positions, cos_sin, H, D, rot, max_pos, status);
}

extern "C" int skein_latent_gather(const void* cache, const int* block_table, int max_blocks, const int* kv_len, const int* q_len,
                                   const int* dense_start, void* dense, int S, int max_ctx, int L, int page_size, int num_pages, int* status,
                                   int fp32, void* stream) {
  using namespace skein;
  if (S == 0 || max_ctx <= 0) return 0;
  const dim3 grid((max_ctx + page_size - 1) / page_size, S);
  if (fp32) return (int)launch_pdl(latent_gather_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)cache, block_table, max_blocks, kv_len, q_len, dense_start, (float*)dense, L, page_size, num_pages, status);
  return (int)launch_pdl(latent_gather_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, (const __nv_bfloat16*)cache, block_table, max_blocks, kv_len, q_len, dense_start, (__nv_bfloat16*)dense, L, page_size, num_pages, status);
}

extern "C" int skein_latent_attn_rows(const void* q_abs, const void* q, long long q_ld, const float* cos_sin, int max_pos, const int* positions,
                                      const int* seq_of_token, const int* block_table, int max_blocks, const void* cache, int num_pages,
                                      int page_size, void* out, int T, int H, int D, int rot, int kv_rank, float scale, const float* sinks, int* status,
                                      int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (rot % 2 != 0 || H > 65535) return -1;
  LatentAttnParams p{q_abs, q, cos_sin, positions, seq_of_token, block_table, cache, out, status, sinks, q_ld, scale, H, D, rot, kv_rank, max_pos,
                     max_blocks, num_pages, page_size};
  const size_t sm = (size_t)(2 * kv_rank + rot + LA_THREADS) * 4;
  if (sm > 200 * 1024) return -1;
  auto go = [&](auto fn) -> int {
    cudaError_t e = sm > 40 * 1024 ? cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm) : cudaSuccess;
    return (int)(e != cudaSuccess ? e : launch_pdl(fn, dim3(T, H), dim3(LA_THREADS), sm, (cudaStream_t)stream, p));
  };
  return fp32 ? go(latent_attn_rows_kernel<float>) : go(latent_attn_rows_kernel<__nv_bfloat16>);
}
