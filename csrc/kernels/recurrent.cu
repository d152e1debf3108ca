// Recurrences with a 32-bit matrix state S [D, V] per head, carried from token to token of a sequence:
//
//   S <- g S + k u^T,   o = S^T q (+ skip v)
//     delta      g = exp(neg_decay softplus(a + dt_bias)),  u = beta (v - (g S)^T k),  beta = sigmoid(b);  q, k unit vectors
//     ssd        g = exp(neg_decay dt),  dt = softplus(dt_raw + dt_bias),  u = dt v
//     lightning  g = exp(neg_decay),  u = v
//
// q, k, v are projections that passed a short causal convolution over time (delta, ssd) and silu. Query / key heads may be
// shared: head h uses h / (H / G).
//
// A sequence owns one slot of the state pools: S [slots, H, D, V] fp32 and the convolution's last inputs [slots, taps, channels]
// in the activation type, position p in row p mod taps (taps - 1 rows would hold the state; with one more, a step writes no row
// it reads). Position 0 starts from zero whatever the slot holds.
//
//   rec_step   decode: one row per sequence. Convolution, silu, unit norms, gates, read-out and update in one kernel
//   rec_prep   chunks: the same up to the gates, for every token of the chunk at once
//   rec_scan   chunks: the recurrence one token after the other (every size and precision; recurrent_tc.cu has the
//              tensor-core form)
//   rec_tail   chunks: the convolution's last inputs into the slot (after every reader of the old ones)
//
// Activations are bf16, or fp32 when a model runs in 32-bit; convolved q, k, v are rounded to the activation type, everything
// after that is 32-bit. Compiled without fast-math.
#include "ptx.cuh"
#include "launch.cuh"
#include "recurrent.cuh"
#include "vec.cuh"
#include <math.h>

namespace skein {

constexpr int RS_THREADS = 256, RS_WARPS = 8;
constexpr int REC_MAX_D = 512;

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// log decay and write coefficient of head h from the row's gate columns
template <typename T>
__device__ __forceinline__ void rec_gates(const RecParams& p, const T* row, int h, float* log_g, float* coef) {
  const float nd = p.neg_decay[h];
  if (p.kind == REC_LIGHTNING) { *log_g = nd; *coef = 1.f; return; }
  const float dt = softplus_f(to_f<T>(row[p.a_col + h]) + p.dt_bias[h]);
  *log_g = nd * dt;
  *coef = p.kind == REC_DELTA ? 1.f / (1.f + expf(-to_f<T>(row[p.b_col + h]))) : dt;
}

// column of the projection row and of the convolution's channel order (q | k | v)
__device__ __forceinline__ int rec_col(const RecParams& p, int ch) {
  const int gd = p.G * p.D;
  return ch < gd ? p.q_col + ch : ch < 2 * gd ? p.k_col + ch - gd : p.v_col + ch - 2 * gd;
}

// Convolution and silu of channel ch of the row at position pos. prev(j): the channel's input j tokens earlier (only asked for
// where it exists).
template <typename T, typename F>
__device__ __forceinline__ float rec_conv(const RecParams& p, int ch, int pos, float cur, F prev) {
  if (p.kind == REC_LIGHTNING) return to_f<T>(from_f<T>(silu_f(cur)));
  float a = p.conv_b ? p.conv_b[ch] : 0.f;
  for (int j = p.taps - 1; j > 0; --j)
    if (pos >= j) a = fmaf(p.conv_w[(size_t)(p.taps - 1 - j) * p.C + ch], prev(j), a);
  a = fmaf(p.conv_w[(size_t)(p.taps - 1) * p.C + ch], cur, a);
  return to_f<T>(from_f<T>(silu_f(a)));
}

// Sums of two values over the CTA, returned to every thread
__device__ __forceinline__ float2 rec_block_sum2(float2 v, float2* sh) {
  for (int o = 16; o > 0; o >>= 1) {
    v.x += __shfl_xor_sync(0xffffffffu, v.x, o);
    v.y += __shfl_xor_sync(0xffffffffu, v.y, o);
  }
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
  __syncthreads();
  float2 t = make_float2(0.f, 0.f);
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) { t.x += sh[i].x; t.y += sh[i].y; }
  return t;
}

// ---- decode -----------------------------------------------------------------------------------------
// grid (column tiles of 32 VPT, H, B). Warp w holds rows w, w + 8, ... of the tile, lane l columns l VPT ...: every warp reads
// whole 32 VPT-wide row pieces. Both products with the old state come from one pass: o = g S^T q + (q . k) u.
template <typename T, int RPT, int VPT>
__global__ void __launch_bounds__(RS_THREADS) rec_step_kernel(const RecParams p) {
  __shared__ float q_s[REC_MAX_D], k_s[REC_MAX_D];
  __shared__ float part[2][RS_WARPS][32 * VPT];
  __shared__ float2 red[RS_WARPS], red2[RS_WARPS];
  __shared__ float v_s[32 * VPT];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pos = p.positions[b];
  if (pos < 0) return;
  const int slot = p.slots[b];
  if (slot < 0 || slot >= p.num_slots) { if (tid == 0) report_status(p.status, ST_BAD_INDEX, slot); return; }
  const int grp = h / (p.H / p.G), tile0 = blockIdx.x * 32 * VPT, c0 = tile0 + lane * VPT;
  float* S = p.state + ((size_t)slot * p.H + h) * p.D * p.V;
  // the state first: its latency covers the convolution
  float s[RPT][VPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int n = warp + i * RS_WARPS;
#pragma unroll
    for (int j = 0; j < VPT; ++j) s[i][j] = 0.f;
    if (n < p.D && c0 < p.V && pos > 0) load_v<float, VPT>(S + (size_t)n * p.V + c0, s[i]);
  }
  const T* row = (const T*)p.row + (size_t)b * p.ld;
  T* tail = p.taps > 1 ? (T*)p.tail + (size_t)slot * p.taps * p.C : nullptr;
  const int gd = p.G * p.D, ncol = min(32 * VPT, p.V - tile0), first_head = grp * (p.H / p.G);
  float2 sq = make_float2(0.f, 0.f);
  for (int i = tid; i < 2 * p.D + ncol; i += RS_THREADS) {
    const int ch = i < p.D ? grp * p.D + i : i < 2 * p.D ? gd + grp * p.D + i - p.D : 2 * gd + h * p.V + tile0 + i - 2 * p.D;
    const float cur = to_f<T>(row[rec_col(p, ch)]);
    const float x = rec_conv<T>(p, ch, pos, cur, [&](int j) { return to_f<T>(tail[(size_t)((pos - j) % p.taps) * p.C + ch]); });
    // one CTA of those that share a channel keeps its input for the next steps
    if (tail && (i >= 2 * p.D || (blockIdx.x == 0 && h == first_head))) tail[(size_t)(pos % p.taps) * p.C + ch] = from_f<T>(cur);
    if (i < p.D) { q_s[i] = x; sq.x += x * x; }
    else if (i < 2 * p.D) { k_s[i - p.D] = x; sq.y += x * x; }
    else v_s[i - 2 * p.D] = x;
  }
  sq = rec_block_sum2(sq, red);      // (also the barrier behind q_s, k_s, v_s)
  float rq = 1.f, rk = 1.f;
  if (p.kind == REC_DELTA) {
    rq = 1.f / sqrtf(sq.x + 1e-6f) / sqrtf((float)p.D);
    rk = 1.f / sqrtf(sq.y + 1e-6f);
  }
  float log_g, coef;
  rec_gates<T>(p, row, h, &log_g, &coef);
  const float g = expf(log_g);
  float qk = 0.f;
  for (int n = tid; n < p.D; n += RS_THREADS) qk += (q_s[n] * rq) * (k_s[n] * rk);
  float ks[VPT], qs[VPT];
#pragma unroll
  for (int j = 0; j < VPT; ++j) ks[j] = qs[j] = 0.f;
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int n = warp + i * RS_WARPS;
    if (n >= p.D) break;
    const float kn = k_s[n] * rk, qn = q_s[n] * rq;
#pragma unroll
    for (int j = 0; j < VPT; ++j) { ks[j] = fmaf(kn, s[i][j], ks[j]); qs[j] = fmaf(qn, s[i][j], qs[j]); }
  }
#pragma unroll
  for (int j = 0; j < VPT; ++j) { part[0][warp][lane * VPT + j] = ks[j]; part[1][warp][lane * VPT + j] = qs[j]; }
  qk = rec_block_sum2(make_float2(qk, 0.f), red2).x;
  float u[VPT];
#pragma unroll
  for (int j = 0; j < VPT; ++j) {
    float a = 0.f, o = 0.f;
#pragma unroll
    for (int w = 0; w < RS_WARPS; ++w) { a += part[0][w][lane * VPT + j]; o += part[1][w][lane * VPT + j]; }
    const bool in = c0 + j < p.V;
    const float v = in ? v_s[lane * VPT + j] : 0.f;
    u[j] = p.kind == REC_DELTA ? coef * (v - g * a) : coef * v;
    if (warp == 0 && in) {
      const float y = g * o + qk * u[j] + (p.skip ? p.skip[h] * v : 0.f);
      ((T*)p.out)[(size_t)b * p.H * p.V + (size_t)h * p.V + c0 + j] = from_f<T>(y);
    }
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int n = warp + i * RS_WARPS;
    if (n >= p.D) break;
    if (c0 >= p.V) continue;
    const float kn = k_s[n] * rk;
#pragma unroll
    for (int j = 0; j < VPT; ++j) s[i][j] = fmaf(g, s[i][j], kn * u[j]);
    store_v<float, VPT>(S + (size_t)n * p.V + c0, s[i]);
  }
}

// ---- chunks ---------------------------------------------------------------------------------------
// grid T. Convolved q | k | v of one token, its heads' gates and (delta) the factors that make q and k unit vectors.
template <typename T>
__global__ void __launch_bounds__(256) rec_prep_kernel(const RecParams p, const RecChunk c) {
  extern __shared__ float qk_s[];        // [2 G D] (delta)
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, pos = p.positions[t];
  const int seq = c.seq_of_token[t], first = c.q_start[seq];
  int slot = p.slots[seq];
  if (slot < 0 || slot >= p.num_slots) { if (tid == 0) report_status(p.status, ST_BAD_INDEX, slot); slot = 0; }
  const T* row = (const T*)p.row + (size_t)t * p.ld;
  const T* tail = p.taps > 1 ? (const T*)p.tail + (size_t)slot * p.taps * p.C : nullptr;
  T* out = (T*)c.qkv + (size_t)t * c.qkv_ld;
  const int gd = p.G * p.D, n = 2 * gd + p.H * p.V;
  for (int ch = tid; ch < n; ch += blockDim.x) {
    const int col = rec_col(p, ch);
    const float x = rec_conv<T>(p, ch, pos, to_f<T>(row[col]), [&](int j) {
      return t - j >= first ? to_f<T>(row[col - (long long)j * p.ld]) : to_f<T>(tail[(size_t)((pos - j) % p.taps) * p.C + ch]);
    });
    out[ch < 2 * gd ? ch : ch - 2 * gd + c.v_off] = from_f<T>(x);
    if (p.kind == REC_DELTA && ch < 2 * gd) qk_s[ch] = x;
  }
  for (int h = tid; h < p.H; h += blockDim.x) {
    float log_g, coef;
    rec_gates<T>(p, row, h, &log_g, &coef);
    c.gates[((size_t)t * p.H + h) * 2] = log_g;
    c.gates[((size_t)t * p.H + h) * 2 + 1] = coef;
  }
  if (p.kind != REC_DELTA) return;
  __syncthreads();
  for (int u = tid >> 5; u < 2 * p.G; u += blockDim.x >> 5) {      // a warp per query / key head
    float ss = 0.f;
    for (int d = tid & 31; d < p.D; d += 32) { const float x = qk_s[(size_t)u * p.D + d]; ss = fmaf(x, x, ss); }
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((tid & 31) == 0) c.unit[(size_t)t * 2 * p.G + u] = 1.f / sqrtf(ss + 1e-6f) / (u < p.G ? sqrtf((float)p.D) : 1.f);
  }
}

// grid S: the last inputs of every channel, position p in row p mod taps
template <typename T>
__global__ void __launch_bounds__(256) rec_tail_kernel(const RecParams p, const RecChunk c) {
  pdl_trigger();
  pdl_wait();
  const int seq = blockIdx.x, len = c.q_len[seq], slot = p.slots[seq];
  if (len < 1 || slot < 0 || slot >= p.num_slots) return;
  const int keep = min(len, p.taps - 1), t_end = c.q_start[seq] + len;
  for (int i = threadIdx.x + blockIdx.y * blockDim.x; i < keep * p.C; i += blockDim.x * gridDim.y) {
    const int ch = i % p.C, t = t_end - 1 - i / p.C;
    ((T*)p.tail)[((size_t)slot * p.taps + p.positions[t] % p.taps) * p.C + ch] = ((const T*)p.row)[(size_t)t * p.ld + rec_col(p, ch)];
  }
}

constexpr int SC_TOK = 16;          // tokens staged at a time
constexpr int SC_COLS = 4;          // columns of a warp: 8 lanes share a column's rows
constexpr int SC_WARPS = 8;

// grid (tiles of 32 columns, H, S). A warp owns 4 columns of the state; lane (r, c) holds rows r, r + 8, ... of column c, so that
// the sums over rows need no more than shuffles.
template <typename T, int RPT>
__global__ void __launch_bounds__(256) rec_scan_kernel(const RecParams p, const RecChunk c) {
  extern __shared__ float sc_s[];      // q [SC_TOK][D], k [SC_TOK][D], v [SC_TOK][32]
  __shared__ float g_s[SC_TOK], coef_s[SC_TOK];
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int len = c.q_len[seq], t0 = c.q_start[seq], slot = p.slots[seq];
  if (len < 1 || slot < 0 || slot >= p.num_slots) return;
  const int grp = h / (p.H / p.G), gd = p.G * p.D, tile0 = blockIdx.x * 32;
  const int r = lane >> 2, col = tile0 + warp * SC_COLS + (lane & 3);
  const bool in = col < p.V;
  float* q_s = sc_s;
  float* k_s = q_s + SC_TOK * p.D;
  float* v_s = k_s + SC_TOK * p.D;
  float* S = p.state + ((size_t)slot * p.H + h) * p.D * p.V;
  const bool fresh = p.positions[t0] == 0;
  float s[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int n = r + 8 * i;
    s[i] = (n < p.D && in && !fresh) ? S[(size_t)n * p.V + col] : 0.f;
  }
  const float skip = p.skip ? p.skip[h] : 0.f;
  for (int b0 = 0; b0 < len; b0 += SC_TOK) {
    const int cnt = min(SC_TOK, len - b0);
    __syncthreads();
    for (int i = tid; i < cnt * p.D; i += 256) {
      const int j = i / p.D, d = i % p.D;
      const T* x = (const T*)c.qkv + (size_t)(t0 + b0 + j) * c.qkv_ld + grp * p.D + d;
      float rq = 1.f, rk = 1.f;
      if (p.kind == REC_DELTA) {
        rq = c.unit[(size_t)(t0 + b0 + j) * 2 * p.G + grp];
        rk = c.unit[(size_t)(t0 + b0 + j) * 2 * p.G + p.G + grp];
      }
      q_s[i] = to_f<T>(x[0]) * rq;
      k_s[i] = to_f<T>(x[gd]) * rk;
    }
    for (int i = tid; i < cnt * 32; i += 256) {
      const int j = i / 32, d = i % 32;
      v_s[i] = tile0 + d < p.V ? to_f<T>(((const T*)c.qkv)[(size_t)(t0 + b0 + j) * c.qkv_ld + c.v_off + h * p.V + tile0 + d]) : 0.f;
    }
    if (tid < cnt) {
      const float* gt = c.gates + ((size_t)(t0 + b0 + tid) * p.H + h) * 2;
      g_s[tid] = expf(gt[0]);
      coef_s[tid] = gt[1];
    }
    __syncthreads();
    for (int j = 0; j < cnt; ++j) {
      const float g = g_s[j], v = v_s[j * 32 + warp * SC_COLS + (lane & 3)];
      float u = coef_s[j] * v;
      if (p.kind == REC_DELTA) {
        float a = 0.f;
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
          const int n = r + 8 * i;
          if (n < p.D) a = fmaf(k_s[j * p.D + n], s[i], a);
        }
        for (int o = 4; o < 32; o <<= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
        u -= coef_s[j] * g * a;
      }
      float o_ = 0.f;
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        const int n = r + 8 * i;
        if (n < p.D) {
          s[i] = fmaf(g, s[i], k_s[j * p.D + n] * u);
          o_ = fmaf(q_s[j * p.D + n], s[i], o_);
        }
      }
      for (int o = 4; o < 32; o <<= 1) o_ += __shfl_xor_sync(0xffffffffu, o_, o);
      if (r == 0 && in) ((T*)p.out)[(size_t)(t0 + b0 + j) * p.H * p.V + (size_t)h * p.V + col] = from_f<T>(o_ + skip * v);
    }
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int n = r + 8 * i;
    if (n < p.D && in) S[(size_t)n * p.V + col] = s[i];
  }
}

template <typename T, int RPT>
static int rec_step_go(const RecParams& p, int B, cudaStream_t s) {
  // whole 128-column tiles when the launch fills the GPU with them, else narrow ones for more CTAs
  const bool wide = RPT <= 16 && p.V % 4 == 0 && (long long)B * p.H * ((p.V + 127) / 128) >= 148;
  if (wide) return (int)launch_pdl(rec_step_kernel<T, (RPT <= 16 ? RPT : 1), 4>, dim3((p.V + 127) / 128, p.H, B), dim3(RS_THREADS), 0, s, p);
  return (int)launch_pdl(rec_step_kernel<T, RPT, 1>, dim3((p.V + 31) / 32, p.H, B), dim3(RS_THREADS), 0, s, p);
}

template <typename T>
static int rec_step_any(const RecParams& p, int B, cudaStream_t s) {
  if (p.D <= 32) return rec_step_go<T, 4>(p, B, s);
  if (p.D <= 64) return rec_step_go<T, 8>(p, B, s);
  if (p.D <= 128) return rec_step_go<T, 16>(p, B, s);
  if (p.D <= 256) return rec_step_go<T, 32>(p, B, s);
  return rec_step_go<T, 64>(p, B, s);
}

template <typename T, int RPT>
static int rec_scan_go(const RecParams& p, const RecChunk& c, int S, cudaStream_t s) {
  const int sm = SC_TOK * (2 * p.D + 32) * 4;
  auto fn = rec_scan_kernel<T, RPT>;
  if (sm > 46 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, sm);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl(fn, dim3((p.V + 31) / 32, p.H, S), dim3(256), (size_t)sm, s, p, c);
}

template <typename T>
static int rec_scan_any(const RecParams& p, const RecChunk& c, int S, cudaStream_t s) {
  if (p.D <= 32) return rec_scan_go<T, 4>(p, c, S, s);
  if (p.D <= 64) return rec_scan_go<T, 8>(p, c, S, s);
  if (p.D <= 128) return rec_scan_go<T, 16>(p, c, S, s);
  if (p.D <= 256) return rec_scan_go<T, 32>(p, c, S, s);
  return rec_scan_go<T, 64>(p, c, S, s);
}

static int rec_check(const RecParams* p) {
  if (p->kind < 0 || p->kind > 2 || p->H < 1 || p->G < 1 || p->H % p->G != 0) return -1;
  if (p->D < 1 || p->D > REC_MAX_D || p->V < 1 || p->taps < 1 || p->H > 65535) return -1;
  if (p->taps > 1 && p->tail == nullptr) return -1;
  return 0;
}

}  // namespace skein

extern "C" int skein_rec_step(const SkeinRecParams* p, int B, int fp32, void* stream) {
  using namespace skein;
  if (B == 0) return 0;
  if (int e = rec_check(p)) return e;
  return fp32 ? rec_step_any<float>(*p, B, (cudaStream_t)stream) : rec_step_any<__nv_bfloat16>(*p, B, (cudaStream_t)stream);
}

extern "C" int skein_rec_prep(const SkeinRecParams* p, const SkeinRecChunk* c, int T, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (int e = rec_check(p)) return e;
  const size_t sm = p->kind == REC_DELTA ? (size_t)2 * p->G * p->D * 4 : 0;
  if (sm > 200 * 1024) return -1;
  auto go = [&](auto fn) -> int {
    if (sm > 46 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
      if (e != cudaSuccess) return (int)e;
    }
    return (int)launch_pdl(fn, dim3(T), dim3(256), sm, (cudaStream_t)stream, *p, *c);
  };
  return fp32 ? go(rec_prep_kernel<float>) : go(rec_prep_kernel<__nv_bfloat16>);
}

extern "C" int skein_rec_scan(const SkeinRecParams* p, const SkeinRecChunk* c, int S, int fp32, void* stream) {
  using namespace skein;
  if (S == 0) return 0;
  if (int e = rec_check(p)) return e;
  return fp32 ? rec_scan_any<float>(*p, *c, S, (cudaStream_t)stream) : rec_scan_any<__nv_bfloat16>(*p, *c, S, (cudaStream_t)stream);
}

extern "C" int skein_rec_tail(const SkeinRecParams* p, const SkeinRecChunk* c, int S, int fp32, void* stream) {
  using namespace skein;
  if (S == 0 || p->taps < 2) return 0;
  const dim3 grid(S, 8);
  return (int)(fp32 ? launch_pdl(rec_tail_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, *p, *c)
                    : launch_pdl(rec_tail_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, *p, *c));
}
