// Grouped-query attention over a window, over chunks or over everything before: the kernels in front of it, and a plain attention kernel
// for every head size and for fp32.
//
//   window_append     per token: q and k divided by the root mean square of all their rows at once, times a weight, the first
//                     rot_dims dimensions of every head rotated (pairs i, i + rot_dims / 2); q back in place, k and v into the
//                     paged cache
//   head_append       per head: bias, RMS norm with a weight, the first rot_dims dimensions rotated (neighbouring pairs, or i and
//                     i + rot_dims / 2), the head divided by its root mean square, each optional; values mixed with another layer's; q back
//                     in place, k and v into the paged cache
//   window_attn_rows  attention of single rows under a SkeinAttnRule (attn_rule.cuh)
//
// Cache page: [kv_heads, page_size, maps * dim] keys, then [kv_heads, page_size, vdim] values (with key and value heads of one width the
// layout of the other attention kernels, [2, kv_heads, page_size, dim]). cos/sin: fp32 table [max_pos, rot_dims / 2, 2] made on the host.
// Compiled without fast-math.
#include "attn_rule.cuh"
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

struct HeadAppendParams {
  void* q;                   // [T, ld] H * maps heads of D; rotated in place
  const void* k;             // [T, ld] K * maps heads of D
  const void* v;             // [T, ld] K heads of V
  const float* cos_sin;      // [max_pos, rot / 2, 2]
  const int* positions;      // [T], -1: padding row
  const int* seq_of_token;   // [T] row of block_table, or null (row = token)
  const int* block_table;    // [S, max_blocks]
  void* cache;               // [pages, K * page_size * (maps * D + V)]
  int* status;
  long long ld;
  int T, H, K, D, maps, V, rot, interleaved, unit, max_pos, max_blocks, num_pages, page_size;
  float eps;
  SkeinHeadExtras x;
};

constexpr int HA_WARPS = 8;

// N elements of a head at element i of it: value, plus the bias
template <typename T, int N>
__device__ __forceinline__ void ha_load(const T* src, const float* bias, int i, float* a) {
  load_v<T, N>(src + i, a);
  if (bias) {
    float b[N];
    load_v<float, N>(bias + i, b);
#pragma unroll
    for (int k = 0; k < N; ++k) a[k] += b[k];
  }
}

// values of a key head: bias, kept for later layers, mixed with the first such layer's
template <typename T, int N>
__device__ __forceinline__ void ha_value(const HeadAppendParams& p, const T* src, T* dst, int t, int n, int i) {
  float a[N];
  const size_t at = (size_t)t * p.K * p.V + (size_t)n * p.V + i;
  ha_load<T, N>(src, p.x.v_bias ? p.x.v_bias + (size_t)n * p.V : nullptr, i, a);
  if (p.x.v_keep) store_v<T, N>((T*)p.x.v_keep + at, a);
  if (p.x.mix) {
    float f[N];
    const float m = p.x.mix[0];
    load_v<T, N>((const T*)p.x.v_first + at, f);
#pragma unroll
    for (int k = 0; k < N; ++k) a[k] = (1.f - m) * a[k] + m * f[k];
  }
  store_v<T, N>(dst + i, a);
}

// One warp per head of a token. PAIR4: neighbouring pairs in accesses of 4 elements (two pairs), else single pairs.
template <typename T, bool PAIR4>
__global__ void __launch_bounds__(32 * HA_WARPS) head_append_kernel(const HeadAppendParams p) {
  pdl_trigger();
  pdl_wait();
  const int nq = p.H * p.maps, nk = p.K * p.maps, units = nq + nk + p.K;
  const long long u = (long long)blockIdx.x * HA_WARPS + (threadIdx.x >> 5);
  if (u >= (long long)p.T * units) return;
  const int t = (int)(u / units), lane = threadIdx.x & 31, pos = p.positions[t];
  int n = (int)(u % units);
  if (pos < 0) return;
  if (pos >= p.max_pos) { if (lane == 0) report_status(p.status, ST_BAD_INDEX, pos); return; }
  const T* src;
  T* dst;
  const float *bias = nullptr, *nw = n < nq ? p.x.q_norm : p.x.k_norm;
  if (n < nq) {
    if (p.x.q_bias) bias = p.x.q_bias + (size_t)n * p.D;
    src = dst = (T*)p.q + (size_t)t * p.ld + (size_t)n * p.D;
  } else {
    const int seq = p.seq_of_token ? p.seq_of_token[t] : t;
    const int page = p.block_table[(size_t)seq * p.max_blocks + pos / p.page_size], slot = pos % p.page_size;
    if (page < 0 || page >= p.num_pages) { if (lane == 0) report_status(p.status, ST_BAD_INDEX, page); return; }
    T* base = (T*)p.cache + (size_t)page * p.K * p.page_size * (p.maps * p.D + p.V);
    n -= nq;
    if (n < nk) {
      if (p.x.k_bias) bias = p.x.k_bias + (size_t)n * p.D;
      src = (const T*)p.k + (size_t)t * p.ld + (size_t)n * p.D;
      dst = base + ((size_t)(n / p.maps) * p.page_size + slot) * p.maps * p.D + (size_t)(n % p.maps) * p.D;
    } else {
      n -= nk;
      src = (const T*)p.v + (size_t)t * p.ld + (size_t)n * p.V;
      dst = base + (size_t)p.K * p.page_size * p.maps * p.D + ((size_t)n * p.page_size + slot) * p.V;
      if (PAIR4 && p.V % 4 == 0) {
        for (int i = lane * 4; i < p.V; i += 128) ha_value<T, 4>(p, src, dst, t, n, i);
      } else {
        for (int i = lane; i < p.V; i += 32) ha_value<T, 1>(p, src, dst, t, n, i);
      }
      return;
    }
  }
  const float2* cs = reinterpret_cast<const float2*>(p.cos_sin) + (size_t)pos * (p.rot / 2);
  if (PAIR4) {
    float r = 1.f;
    if (p.unit || nw) {      // a rotation leaves the sum of squares as it is
      float ss = 0.f;
      for (int i = lane * 4; i < p.D; i += 128) {
        float a[4];
        ha_load<T, 4>(src, bias, i, a);
#pragma unroll
        for (int k = 0; k < 4; ++k) ss = fmaf(a[k], a[k], ss);
      }
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      r = 1.f / sqrtf(ss / (float)p.D + p.eps);
    }
    for (int i = lane * 4; i < p.D; i += 128) {
      float a[4];
      ha_load<T, 4>(src, bias, i, a);
      if (nw) {
        float w[4];
        load_v<float, 4>(nw + i, w);
#pragma unroll
        for (int k = 0; k < 4; ++k) a[k] *= w[k];
      }
      if (i < p.rot) {
        const float4 c = *reinterpret_cast<const float4*>(cs + i / 2);
        const float x0 = a[0], x2 = a[2];
        a[0] = x0 * c.x - a[1] * c.y; a[1] = a[1] * c.x + x0 * c.y;
        a[2] = x2 * c.z - a[3] * c.w; a[3] = a[3] * c.z + x2 * c.w;
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) a[k] *= r;
      store_v<T, 4>(dst + i, a);
    }
    return;
  }
  float r = 1.f;
  auto value = [&](int i) { return to_f<T>(src[i]) + (bias ? bias[i] : 0.f); };
  auto weight = [&](int i) { return nw ? nw[i] : 1.f; };
  if (p.unit || nw) {
    float ss = 0.f;
    for (int i = lane; i < p.D; i += 32) { const float a = value(i); ss = fmaf(a, a, ss); }
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    r = 1.f / sqrtf(ss / (float)p.D + p.eps);
  }
  const int half = p.rot / 2;
  for (int i = lane; i < half; i += 32) {
    const int i0 = p.interleaved ? 2 * i : i, i1 = p.interleaved ? 2 * i + 1 : i + half;
    const float2 c = cs[i];
    const float x = value(i0) * weight(i0), y = value(i1) * weight(i1);
    dst[i0] = from_f<T>((x * c.x - y * c.y) * r);
    dst[i1] = from_f<T>((y * c.x + x * c.y) * r);
  }
  for (int i = p.rot + lane; i < p.D; i += 32) dst[i] = from_f<T>(value(i) * weight(i) * r);
}

struct WindowAttnParams {
  const void* q;             // [T, ld] rotated queries, maps * D per head
  const void* cache;
  const int* positions;
  const int* seq_of_token;
  const int* block_table;
  void* out;                 // [T, out_ld] heads * vdim columns
  int* status;
  long long ld, out_ld;
  int H, K, D, V, max_blocks, num_pages, page_size;
  SkeinAttnRule r;
};

constexpr int WR_TILE = 128;       // keys per round, one per thread

// grid (T, H), 128 threads. Per map: scores of a tile of keys, running softmax, then every thread sums the values of its output columns.
template <typename T>
__global__ void __launch_bounds__(WR_TILE) window_attn_rows_kernel(const WindowAttnParams p) {
  extern __shared__ float q_s[];           // [D] query, then [maps][V] sums
  __shared__ float prob[WR_TILE];
  __shared__ const T* page_s[WR_TILE];
  __shared__ float red[4];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, pos = p.positions[t], maps = p.r.maps;
  if (pos < 0) return;
  const int kvh = h / (p.H / p.K), seq = p.seq_of_token ? p.seq_of_token[t] : t;
  const int lo = attn_first_key(p.r.window, p.r.chunk, pos), KW = maps * p.D;
  const int kept = min(p.r.keep_first, lo), n_keys = kept + pos + 1 - lo;      // the first tokens, then the window
  const size_t page_elems = (size_t)p.K * p.page_size * (KW + p.V);
  for (int map = 0; map < maps; ++map) {
    float* o_s = q_s + p.D + map * p.V;
    const T* q = (const T*)p.q + (size_t)t * p.ld + (size_t)h * KW + (size_t)map * p.D;
    __syncthreads();
    for (int i = tid; i < p.D; i += WR_TILE) q_s[i] = to_f<T>(q[i]);
    for (int i = tid; i < p.V; i += WR_TILE) o_s[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int i0 = 0; i0 < n_keys; i0 += WR_TILE) {
      __syncthreads();
      const int cnt = min(WR_TILE, n_keys - i0), j = i0 + tid < kept ? i0 + tid : i0 + tid - kept + lo;
      float s = -INFINITY;
      if (tid < cnt) {
        int page = p.block_table[(size_t)seq * p.max_blocks + j / p.page_size];
        if (page < 0 || page >= p.num_pages) { report_status(p.status, ST_BAD_INDEX, page); page = 0; }
        const T* base = (const T*)p.cache + (size_t)page * page_elems;
        const T* k = base + ((size_t)kvh * p.page_size + j % p.page_size) * KW + (size_t)map * p.D;
        page_s[tid] = base + (size_t)p.K * p.page_size * KW + ((size_t)kvh * p.page_size + j % p.page_size) * p.V;
        float a = 0.f;
        for (int d = 0; d < p.D; ++d) a = fmaf(q_s[d], to_f<T>(k[d]), a);
        s = a * p.r.scale;
        if (p.r.softcap > 0.f) s = p.r.softcap * tanhf(s / p.r.softcap);
      }
      float mx = s;
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      if ((tid & 31) == 0) red[tid >> 5] = mx;
      __syncthreads();
      const float mn = fmaxf(m, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
      const float keep = m == -INFINITY ? 0.f : expf(m - mn), e = tid < cnt ? expf(s - mn) : 0.f;
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
    float inv = 1.f / l;
    if (p.r.sink || p.r.sinks) {
      const float sink = p.r.sinks ? p.r.sinks[h] : 0.f, top = fmaxf(m, sink), e = expf(m - top);
      inv = e / (l * e + expf(sink - top));
    }
    for (int d = tid; d < p.V; d += WR_TILE) o_s[d] *= inv;
  }
  const float* o = q_s + p.D;              // (a thread reads what it wrote)
  float f = p.r.out_scale;
  if (maps == 2) {
    const float lam = p.r.lam[0];
    float ss = 0.f;
    for (int d = tid; d < p.V; d += WR_TILE) { const float a = o[d] - lam * o[p.V + d]; ss = fmaf(a, a, ss); }
    for (int k = 16; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
    __syncthreads();
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    f /= sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)p.V + p.r.eps);
  }
  T* out = (T*)p.out + (size_t)t * p.out_ld + (size_t)h * p.V;
  const T* gate = p.r.gate ? (const T*)p.r.gate + (size_t)t * p.r.gate_ld + (size_t)h * p.V : nullptr;
  for (int d = tid; d < p.V; d += WR_TILE) {
    float a = maps == 2 ? o[d] - p.r.lam[0] * o[p.V + d] : o[d];
    a *= f;
    if (gate) a /= 1.f + expf(-to_f<T>(gate[d]));
    out[d] = from_f<T>(a);
  }
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

extern "C" int skein_head_append(void* q, const void* k, const void* v, long long ld, const float* cos_sin, const int* positions,
                                 const int* seq_of_token, const int* block_table, void* cache, int* status, const SkeinHeadExtras* extras, int T, int H,
                                 int K, int D, int maps, int V,
                                 int rot, int interleaved, int unit, int max_pos, int max_blocks, int num_pages, int page_size, float eps, int fp32,
                                 void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (rot % 2 != 0 || rot > D || rot < 0 || (rot > 0 && !cos_sin) || (extras->mix && !extras->v_first)) return -1;
  HeadAppendParams p{q, k, v, cos_sin, positions, seq_of_token, block_table, cache, status, ld, T, H, K, D, maps, V, rot, interleaved, unit, max_pos,
                     max_blocks, num_pages, page_size, eps, *extras};
  const bool v4 = (interleaved || rot == 0) && D % 4 == 0 && rot % 4 == 0 && V % 4 == 0 && ld % 4 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)k % 16 == 0 &&
                  (uintptr_t)v % 16 == 0 && (uintptr_t)cache % 16 == 0;
  const long long units = (long long)T * (H * maps + K * maps + K);
  const dim3 grid((unsigned)((units + HA_WARPS - 1) / HA_WARPS)), b(32 * HA_WARPS);
  cudaStream_t s = (cudaStream_t)stream;
  if (fp32) return (int)(v4 ? launch_pdl(head_append_kernel<float, true>, grid, b, 0, s, p) : launch_pdl(head_append_kernel<float, false>, grid, b, 0, s, p));
  return (int)(v4 ? launch_pdl(head_append_kernel<__nv_bfloat16, true>, grid, b, 0, s, p)
                  : launch_pdl(head_append_kernel<__nv_bfloat16, false>, grid, b, 0, s, p));
}

extern "C" int skein_window_attn_rows(const void* q, long long ld, const void* cache, const int* positions, const int* seq_of_token,
                                      const int* block_table, void* out, long long out_ld, int* status, int T, int H, int K, int D, int V, int max_blocks,
                                      int num_pages, int page_size, const SkeinAttnRule* rule, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (H % K != 0 || rule->maps < 1 || rule->maps > 2 || (rule->maps == 2 && !rule->lam) || (D + rule->maps * V) * 4 > 40 * 1024) return -1;
  WindowAttnParams p{q, cache, positions, seq_of_token, block_table, out, status, ld, out_ld, H, K, D, V, max_blocks, num_pages, page_size, *rule};
  const dim3 grid(T, H);
  const size_t sm = (size_t)(D + rule->maps * V) * 4;
  cudaStream_t s = (cudaStream_t)stream;
  return (int)(fp32 ? launch_pdl(window_attn_rows_kernel<float>, grid, dim3(WR_TILE), sm, s, p)
                    : launch_pdl(window_attn_rows_kernel<__nv_bfloat16>, grid, dim3(WR_TILE), sm, s, p));
}
