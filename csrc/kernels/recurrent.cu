// Recurrences with a 32-bit matrix state S [D, V] per head, carried from token to token of a sequence:
//
//   S <- g S + k u^T,   o = S^T q (+ skip v)
//     delta      g = exp(neg_decay softplus(a + dt_bias)),  u = beta (v - (g S)^T k),  beta = sigmoid(b);  q, k unit vectors
//     channel    the same with one g per row of S: g[n] = exp(neg_decay softplus(step[n] + dt_bias[n]))
//     ssd        g = exp(neg_decay dt),  dt = softplus(dt_raw + dt_bias),  u = dt v
//     lightning  g fixed per head (neg_decay its logarithm),  u = v
//
// q, k, v are projections that passed a short causal convolution over time (delta, ssd) and silu. Query / key heads may be
// shared: head h uses h / (H / G). A decay just below one is raised to a high power in the end: decays per row enter as s + expm1(log g) s.
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
#include "act.cuh"
#include "ptx.cuh"
#include "launch.cuh"
#include "recurrent.cuh"
#include "vec.cuh"
#include <math.h>

namespace skein {

constexpr int RS_THREADS = 256, RS_WARPS = 8;
constexpr int REC_MAX_D = 512;

// log decay and write coefficient of head h from the row's gate columns
template <typename T>
__device__ __forceinline__ void rec_gates(const RecParams& p, const T* row, int h, float* log_g, float* coef) {
  const float nd = p.neg_decay[h];
  if (p.kind == REC_CHANNEL) { *log_g = 0.f; *coef = 1.f / (1.f + expf(-to_f<T>(row[p.b_col + h]))); return; }      // (decays: rec_row_decay)
  if (p.kind == REC_LIGHTNING) { *log_g = nd; *coef = 1.f; return; }
  const float dt = softplus_f(to_f<T>(row[p.a_col + h]) + p.dt_bias[h]);
  *log_g = nd * dt;
  *coef = p.kind == REC_DELTA ? 1.f / (1.f + expf(-to_f<T>(row[p.b_col + h]))) : dt;
}

// g - 1 of row n of head h's state (channel) for the step's row t
__device__ __forceinline__ float rec_row_decay(const RecParams& p, size_t t, int h, int n) {
  const int i = h * p.D + n;
  return expm1f(p.neg_decay[h] * softplus_f(p.step[t * p.H * p.D + i] + p.dt_bias[i]));
}

// column of the projection row and of the convolution's channel order (q | k | v)
__device__ __forceinline__ int rec_col(const RecParams& p, int ch) {
  const int gd = p.G * p.D;
  return ch < gd ? p.q_col + ch : ch < 2 * gd ? p.k_col + ch - gd : p.v_col + ch - 2 * gd;
}

// Convolution and silu of channel ch of the row at position pos. prev(j): the channel's input j tokens earlier (only asked for
// where it exists). TAPS 0: any number.
template <typename T, int TAPS, typename F>
__device__ __forceinline__ float rec_conv(const RecParams& p, int ch, int pos, float cur, F prev) {
  if (p.kind == REC_LIGHTNING) return to_f<T>(from_f<T>(silu_act<T>(cur)));
  float a = p.conv_b ? p.conv_b[ch] : 0.f;
  if (TAPS > 0) {
    float x[TAPS > 0 ? TAPS : 1], w[TAPS > 0 ? TAPS : 1];
#pragma unroll
    for (int j = TAPS - 1; j > 0; --j) {
      x[j] = pos >= j ? prev(j) : 0.f;
      w[j] = p.conv_w[(size_t)(TAPS - 1 - j) * p.C + ch];
    }
#pragma unroll
    for (int j = TAPS - 1; j > 0; --j) a = fmaf(w[j], x[j], a);
  } else {
    for (int j = p.taps - 1; j > 0; --j)
      if (pos >= j) a = fmaf(p.conv_w[(size_t)(p.taps - 1 - j) * p.C + ch], prev(j), a);
  }
  a = fmaf(p.conv_w[(size_t)(p.taps - 1) * p.C + ch], cur, a);
  return to_f<T>(from_f<T>(silu_act<T>(a)));
}

// row of the convolution's cache that holds the input j tokens before position pos (at = pos mod taps)
__device__ __forceinline__ int rec_tail_row(int at, int j, int taps) { return at >= j ? at - j : at - j + taps; }

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
  __shared__ float q_s[REC_MAX_D], k_s[REC_MAX_D], g_s[REC_MAX_D];
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
  if (p.kind == REC_CHANNEL) for (int n = tid; n < p.D; n += RS_THREADS) g_s[n] = rec_row_decay(p, b, h, n);
  float2 sq = make_float2(0.f, 0.f);
  for (int i = tid; i < 2 * p.D + ncol; i += RS_THREADS) {
    const int ch = i < p.D ? grp * p.D + i : i < 2 * p.D ? gd + grp * p.D + i - p.D : 2 * gd + h * p.V + tile0 + i - 2 * p.D;
    const float cur = to_f<T>(row[rec_col(p, ch)]);
    const float x = rec_conv<T, 0>(p, ch, pos, cur, [&](int j) { return to_f<T>(tail[(size_t)((pos - j) % p.taps) * p.C + ch]); });
    // one CTA of those that share a channel keeps its input for the next steps
    if (tail && (i >= 2 * p.D || (blockIdx.x == 0 && h == first_head))) tail[(size_t)(pos % p.taps) * p.C + ch] = from_f<T>(cur);
    if (i < p.D) { q_s[i] = x; sq.x += x * x; }
    else if (i < 2 * p.D) { k_s[i - p.D] = x; sq.y += x * x; }
    else v_s[i - 2 * p.D] = x;
  }
  sq = rec_block_sum2(sq, red);      // (also the barrier behind q_s, k_s, v_s)
  float rq = 1.f, rk = 1.f;
  if (rec_corrects(p.kind)) {
    rq = 1.f / sqrtf(sq.x + 1e-6f) / sqrtf((float)p.D);
    rk = 1.f / sqrtf(sq.y + 1e-6f);
  }
  float log_g, coef;
  rec_gates<T>(p, row, h, &log_g, &coef);
  const float g = p.decay ? p.decay[h] : expf(log_g);
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
    if (p.kind == REC_CHANNEL) {
#pragma unroll
      for (int j = 0; j < VPT; ++j) s[i][j] = fmaf(g_s[n], s[i][j], s[i][j]);
    }
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
    u[j] = rec_corrects(p.kind) ? coef * (v - g * a) : coef * v;
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

// The same with the head's whole state (a contiguous block of up to RSB_MAX bytes) brought to shared memory by one bulk copy: few
// registers, so that three CTAs fit an SM and one's copy runs behind the others' arithmetic. Thread (c, r): columns 4c .. 4c + 3, rows
// r, r + R, ... with R = 1024 / V. V a power of two from 32 to 256. A CTA takes `heads` heads of a group, whose states lie one after
// another and whose queries and keys are the same. grid (H / heads, B).
constexpr int RSB_MAX = 64 * 1024, RSB_HEADS = 8;

template <typename T, int TAPS, bool CHANNEL>
__global__ void __launch_bounds__(RS_THREADS) rec_step_bulk_kernel(const RecParams p, const RecGate gt, const int heads) {
  // states [heads][D][V], then u [V], sums [warps][V], v [heads][V], q [D], k [D], decays [heads][D] (channel)
  extern __shared__ __align__(128) float st_s[];
  float* u_s = st_s + heads * p.D * p.V;
  float* part = u_s + p.V;
  float* v_s = part + RS_WARPS * p.V;
  float* q_s = v_s + heads * p.V;
  float* k_s = q_s + p.D;
  float* g_s = k_s + p.D;
  __shared__ float2 red[RS_WARPS], red2[RS_WARPS];
  __shared__ float2 gate_s[RSB_HEADS];
  __shared__ __align__(8) uint64_t bar;
  __shared__ int gone;
  pdl_trigger();
  pdl_wait();
  const int h0 = blockIdx.x * heads, b = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pos = p.positions[b];
  if (pos < 0) return;
  const int slot = p.slots[b];
  if (slot < 0 || slot >= p.num_slots) { if (tid == 0) report_status(p.status, ST_BAD_INDEX, slot); return; }
  const int D = p.D, V = p.V, grp = h0 / (p.H / p.G);
  float* S = p.state + ((size_t)slot * p.H + h0) * D * V;
  if (tid == 0) {
    gone = 0;
    mbar_init(smem_u32(&bar), 1);
    fence_mbar_init();
    if (pos > 0) {
      mbar_expect_tx(smem_u32(&bar), (uint32_t)(heads * D * V * 4));
      bulk_load_1d(smem_u32(st_s), S, (uint32_t)(heads * D * V * 4), smem_u32(&bar));
    }
  }
  const T* row = (const T*)p.row + (size_t)b * p.ld;
  T* tail = p.taps > 1 ? (T*)p.tail + (size_t)slot * p.taps * p.C : nullptr;
  const int gd = p.G * D;
  if (warp == RS_WARPS - 1 && lane < heads) {
    float log_g, coef;
    rec_gates<T>(p, row, h0 + lane, &log_g, &coef);
    gate_s[lane] = make_float2(p.decay ? p.decay[h0 + lane] : expf(log_g), coef);
  }
  if (CHANNEL) for (int i = tid; i < heads * D; i += RS_THREADS) g_s[i] = rec_row_decay(p, b, h0 + i / D, i % D);
  float2 sq = make_float2(0.f, 0.f);
  const int at = p.taps > 1 ? pos % p.taps : 0;
  const bool owner = h0 % (p.H / p.G) == 0;      // of the group's queries and keys
#pragma unroll 2
  for (int i = tid; i < 2 * D + heads * V; i += RS_THREADS) {
    const int ch = i < D ? grp * D + i : i < 2 * D ? gd + grp * D + i - D : 2 * gd + h0 * V + i - 2 * D;
    const float cur = to_f<T>(row[rec_col(p, ch)]);
    const float x = rec_conv<T, TAPS>(p, ch, pos, cur, [&](int j) { return to_f<T>(tail[(size_t)rec_tail_row(at, j, p.taps) * p.C + ch]); });
    if (tail && (i >= 2 * D || owner)) tail[(size_t)at * p.C + ch] = from_f<T>(cur);
    if (i < D) { q_s[i] = x; sq.x += x * x; }
    else if (i < 2 * D) { k_s[i - D] = x; sq.y += x * x; }
    else v_s[i - 2 * D] = x;
  }
  sq = rec_block_sum2(sq, red);      // (also the barrier behind what was written above)
  float rq = 1.f, rk = 1.f;
  if (rec_corrects(p.kind)) {
    rq = 1.f / sqrtf(sq.x + 1e-6f) / sqrtf((float)D);
    rk = 1.f / sqrtf(sq.y + 1e-6f);
  }
  float qk = 0.f;
  for (int n = tid; n < D; n += RS_THREADS) qk = fmaf(q_s[n], k_s[n], qk);
  qk = rec_block_sum2(make_float2(qk, 0.f), red2).x * rq * rk;
  if (pos > 0) {
    if (!mbar_wait(smem_u32(&bar), 0, &gone, 2000000000ull)) { if (tid == 0) report_status(p.status, ST_TIMEOUT_SMEM_FULL, 30); return; }
  } else {
    for (int i = tid; i < heads * D * V; i += RS_THREADS) st_s[i] = 0.f;
    __syncthreads();
  }
  const int CG = V / 4, R = RS_THREADS / CG, cg = tid % CG, r0 = tid / CG;
  // sums per warp, or (V = 256) per pair of warps that share the columns' halves
  const int pr = CG <= 32 ? warp : r0, np = CG <= 32 ? RS_WARPS : R;
  for (int hh = 0; hh < heads; ++hh) {
    const int h = h0 + hh;
    float* st = st_s + hh * D * V;
    const float g = gate_s[hh].x, coef = gate_s[hh].y;
    const float* gr = g_s + hh * D;
    auto row_of = [&](int n) {      // the state's row, decayed (channel)
      float4 s = *reinterpret_cast<const float4*>(st + n * V + cg * 4);
      if (CHANNEL) {
        const float d = gr[n];
        s.x = fmaf(d, s.x, s.x); s.y = fmaf(d, s.y, s.y); s.z = fmaf(d, s.z, s.z); s.w = fmaf(d, s.w, s.w);
      }
      return s;
    };
    float4 ks = make_float4(0.f, 0.f, 0.f, 0.f), qs = ks;
#pragma unroll 4
    for (int n = r0; n < D; n += R) {
      const float4 s = row_of(n);
      const float kn = k_s[n], qn = q_s[n];
      ks.x = fmaf(kn, s.x, ks.x); ks.y = fmaf(kn, s.y, ks.y); ks.z = fmaf(kn, s.z, ks.z); ks.w = fmaf(kn, s.w, ks.w);
      qs.x = fmaf(qn, s.x, qs.x); qs.y = fmaf(qn, s.y, qs.y); qs.z = fmaf(qn, s.z, qs.z); qs.w = fmaf(qn, s.w, qs.w);
    }
    for (int o = CG; o < 32; o <<= 1) {      // several row groups in a warp
      ks.x += __shfl_xor_sync(0xffffffffu, ks.x, o); ks.y += __shfl_xor_sync(0xffffffffu, ks.y, o);
      ks.z += __shfl_xor_sync(0xffffffffu, ks.z, o); ks.w += __shfl_xor_sync(0xffffffffu, ks.w, o);
      qs.x += __shfl_xor_sync(0xffffffffu, qs.x, o); qs.y += __shfl_xor_sync(0xffffffffu, qs.y, o);
      qs.z += __shfl_xor_sync(0xffffffffu, qs.z, o); qs.w += __shfl_xor_sync(0xffffffffu, qs.w, o);
    }
    const bool writes = CG > 32 || lane < CG;
    float a = 0.f, y = 0.f;
    if (rec_corrects(p.kind)) {              // only the correction needs S^T k
      if (writes) *reinterpret_cast<float4*>(part + pr * V + cg * 4) = ks;
      __syncthreads();
      if (tid < V) for (int w = 0; w < np; ++w) a += part[w * V + tid];
      __syncthreads();
    }
    if (writes) *reinterpret_cast<float4*>(part + pr * V + cg * 4) = qs;
    __syncthreads();
    float o = 0.f;
    if (tid < V) {
      for (int w = 0; w < np; ++w) y += part[w * V + tid];
      const float v = v_s[hh * V + tid];
      const float u = rec_corrects(p.kind) ? coef * (v - g * rk * a) : coef * v;
      u_s[tid] = u * rk;
      o = g * rq * y + qk * u + (p.skip ? p.skip[h] * v : 0.f);
      if (gt.out == nullptr) ((T*)p.out)[(size_t)b * p.H * V + (size_t)h * V + tid] = from_f<T>(o);
    }
    if (gt.out != nullptr) {
      // the head's own norm and gate
      const float r = 1.f / sqrtf(rec_block_sum2(make_float2(o * o, 0.f), red).x / (float)V + gt.eps);      // (a barrier behind u_s too)
      if (tid < V) {
        const float z = to_f<T>(((const T*)gt.gate)[(size_t)b * gt.gate_ld + (size_t)h * V + tid]), a = (gt.sigmoid ? 1.f : z) / (1.f + expf(-z));
        ((T*)gt.out)[(size_t)b * gt.out_ld + (size_t)h * V + tid] = from_f<T>(o * r * gt.norm[tid] * a * gt.scale);
      }
    } else {
      __syncthreads();
    }
    const float4 u4 = *reinterpret_cast<const float4*>(u_s + cg * 4);
#pragma unroll 4
    for (int n = r0; n < D; n += R) {
      float4 s = row_of(n);
      const float kn = k_s[n];
      s.x = fmaf(g, s.x, kn * u4.x); s.y = fmaf(g, s.y, kn * u4.y); s.z = fmaf(g, s.z, kn * u4.z); s.w = fmaf(g, s.w, kn * u4.w);
      *reinterpret_cast<float4*>(S + (size_t)hh * D * V + (size_t)n * V + cg * 4) = s;
    }
    if (hh + 1 < heads) __syncthreads();     // u, the sums and the reduction's scratch are used again
  }
}

template <typename T, int TAPS, bool CHANNEL>
static int rec_step_bulk_go(const RecParams& p, const RecGate& g, int B, cudaStream_t s) {
  int heads = RSB_HEADS;                     // a power of two that divides the heads of a group; enough CTAs before larger ones
  while (heads > 1 && ((p.H / p.G) % heads != 0 || (long long)heads * p.D * p.V * 4 > RSB_MAX || (long long)B * p.H / heads < 444)) heads /= 2;
  const int sm = (heads * p.D * p.V + (RS_WARPS + 1 + heads) * p.V + (2 + (CHANNEL ? heads : 0)) * p.D) * 4;
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(rec_step_bulk_kernel<T, TAPS, CHANNEL>, cudaFuncAttributeMaxDynamicSharedMemorySize, RSB_MAX + 24 * 1024);
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  return (int)launch_pdl(rec_step_bulk_kernel<T, TAPS, CHANNEL>, dim3(p.H / heads, B), dim3(RS_THREADS), (size_t)sm, s, p, g, heads);
}

template <typename T, bool CHANNEL>
static int rec_step_bulk_taps(const RecParams& p, const RecGate& g, int B, cudaStream_t s) {
  switch (p.taps) {
    case 1: return rec_step_bulk_go<T, 1, CHANNEL>(p, g, B, s);
    case 2: return rec_step_bulk_go<T, 2, CHANNEL>(p, g, B, s);
    case 3: return rec_step_bulk_go<T, 3, CHANNEL>(p, g, B, s);
    case 4: return rec_step_bulk_go<T, 4, CHANNEL>(p, g, B, s);
    default: return rec_step_bulk_go<T, 0, CHANNEL>(p, g, B, s);
  }
}

template <typename T>
static int rec_step_bulk(const RecParams& p, const RecGate& g, int B, cudaStream_t s) {
  return p.kind == REC_CHANNEL ? rec_step_bulk_taps<T, true>(p, g, B, s) : rec_step_bulk_taps<T, false>(p, g, B, s);
}

// ---- chunks ---------------------------------------------------------------------------------------
// grid T. Convolved q | k | v of one token, its heads' gates and (delta rules) the factors that make q and k unit vectors.
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
    const float x = rec_conv<T, 0>(p, ch, pos, to_f<T>(row[col]), [&](int j) {
      return t - j >= first ? to_f<T>(row[col - (long long)j * p.ld]) : to_f<T>(tail[(size_t)((pos - j) % p.taps) * p.C + ch]);
    });
    out[ch < 2 * gd ? ch : ch - 2 * gd + c.v_off] = from_f<T>(x);
    if (rec_corrects(p.kind) && ch < 2 * gd) qk_s[ch] = x;
  }
  for (int h = tid; h < p.H; h += blockDim.x) {
    float log_g, coef;
    rec_gates<T>(p, row, h, &log_g, &coef);
    c.gates[((size_t)t * p.H + h) * 2] = log_g;
    c.gates[((size_t)t * p.H + h) * 2 + 1] = coef;
  }
  if (!rec_corrects(p.kind)) return;
  __syncthreads();
  for (int u = tid >> 5; u < 2 * p.G; u += blockDim.x >> 5) {      // a warp per query / key head
    float ss = 0.f;
    for (int d = tid & 31; d < p.D; d += 32) { const float x = qk_s[(size_t)u * p.D + d]; ss = fmaf(x, x, ss); }
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((tid & 31) == 0) c.unit[(size_t)t * 2 * p.G + u] = 1.f / sqrtf(ss + 1e-6f) / (u < p.G ? sqrtf((float)p.D) : 1.f);
  }
}

// The same with 16-byte accesses: a thread takes 8 channels of PV_TOK tokens and keeps the sums of the next TAPS outputs in registers,
// into which every input goes as it is read. Every section starts at a multiple of 8 channels and columns; D / 8 is a power of two up
// to 32 (delta). The last column of CTAs does the gates. grid (channel blocks + 1, token blocks)
constexpr int PV_TOK = 32, PV_AHEAD = 4;       // tokens of a thread; loads in flight

__device__ __forceinline__ float bf_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf_hi(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }
__device__ __forceinline__ uint32_t bf_pack(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ void bf_unpack8(const uint4& u, float* v) {
  v[0] = bf_lo(u.x); v[1] = bf_hi(u.x); v[2] = bf_lo(u.y); v[3] = bf_hi(u.y);
  v[4] = bf_lo(u.z); v[5] = bf_hi(u.z); v[6] = bf_lo(u.w); v[7] = bf_hi(u.w);
}

template <int TAPS>      // 1: no convolution ("lightning"), else the taps
__global__ void __launch_bounds__(256, 2) rec_prep_vec_kernel(const RecParams p, const RecChunk c, int T) {
  __shared__ int pos_s[PV_TOK], first_s[PV_TOK], slot_s[PV_TOK];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, t0 = blockIdx.y * PV_TOK, nt = min(PV_TOK, T - t0);
  if ((int)blockIdx.x == (int)gridDim.x - 1) {
    for (int i = tid; i < nt * p.H; i += 256) {
      const int t = t0 + i / p.H, h = i % p.H;
      float log_g, coef;
      rec_gates<__nv_bfloat16>(p, (const __nv_bfloat16*)p.row + (size_t)t * p.ld, h, &log_g, &coef);
      reinterpret_cast<float2*>(c.gates)[(size_t)t * p.H + h] = make_float2(log_g, coef);
    }
    return;
  }
  if (tid < nt) {
    const int t = t0 + tid, seq = c.seq_of_token[t];
    int slot = p.slots[seq];
    if (slot < 0 || slot >= p.num_slots) { report_status(p.status, ST_BAD_INDEX, slot); slot = 0; }
    pos_s[tid] = p.positions[t];
    first_s[tid] = c.q_start[seq];
    slot_s[tid] = slot;
  }
  __syncthreads();
  const int gd = p.G * p.D, n8 = (2 * gd + p.H * p.V) / 8, g8 = blockIdx.x * 256 + tid;
  const bool live = g8 < n8;
  const int ch = (live ? g8 : 0) * 8, col = rec_col(p, ch);
  const __nv_bfloat16* src = (const __nv_bfloat16*)p.row + (size_t)t0 * p.ld + col;
  __nv_bfloat16* dst = (__nv_bfloat16*)c.qkv + (size_t)t0 * c.qkv_ld + (ch < 2 * gd ? ch : ch - 2 * gd + c.v_off);
  // w[j]: the tap j tokens back. sum[j] (j > 0): what the inputs so far add to the output j - 1 tokens on; the bias is in it
  float w[TAPS][8], bias[8], sum[TAPS][8];
  if (TAPS > 1) {
#pragma unroll
    for (int k = 0; k < 8; ++k) bias[k] = p.conv_b ? p.conv_b[ch + k] : 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      load_v<float, 4>(p.conv_w + (size_t)(TAPS - 1 - j) * p.C + ch, w[j]);
      load_v<float, 4>(p.conv_w + (size_t)(TAPS - 1 - j) * p.C + ch + 4, w[j] + 4);
    }
  }
  const int lanes = p.D / 8;
  const bool units = rec_corrects(p.kind) && blockIdx.x * 2048 < 2 * gd;
  auto token = [&](int i, const uint4& in) {
    float x[8], y[8];
    if (TAPS > 1) {
      const int t = t0 + i, first = first_s[i], pos = pos_s[i];
      if (i == 0 || t == first) {
        // start of the block or of a sequence: the inputs before it, from the chunk, from the cache, or none
#pragma unroll
        for (int j = 1; j < TAPS; ++j)
#pragma unroll
          for (int k = 0; k < 8; ++k) sum[j][k] = bias[k];
#pragma unroll
        for (int j = 1; j < TAPS; ++j) {
          uint4 u = make_uint4(0, 0, 0, 0);
          if (t - j >= first) u = *reinterpret_cast<const uint4*>(src + (long long)(i - j) * p.ld);
          else if (pos - j >= 0)
            u = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)p.tail + ((size_t)slot_s[i] * TAPS + (pos - j) % TAPS) * p.C + ch);
          bf_unpack8(u, x);
#pragma unroll
          for (int o = 0; o + j < TAPS; ++o)        // the output o tokens on sees this input o + j back
#pragma unroll
            for (int k = 0; k < 8; ++k) sum[o + 1][k] = fmaf(w[o + j][k], x[k], sum[o + 1][k]);
        }
      }
      bf_unpack8(in, x);
#pragma unroll
      for (int k = 0; k < 8; ++k) y[k] = fmaf(w[0][k], x[k], sum[1][k]);
#pragma unroll
      for (int j = 1; j + 1 < TAPS; ++j)
#pragma unroll
        for (int k = 0; k < 8; ++k) sum[j][k] = fmaf(w[j][k], x[k], sum[j + 1][k]);
#pragma unroll
      for (int k = 0; k < 8; ++k) sum[TAPS - 1][k] = fmaf(w[TAPS - 1][k], x[k], bias[k]);
    } else {
      bf_unpack8(in, y);
    }
    uint32_t o[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) o[k] = bf_pack(silu_act<__nv_bfloat16>(y[2 * k]), silu_act<__nv_bfloat16>(y[2 * k + 1]));
    if (live) *reinterpret_cast<uint4*>(dst + (long long)i * c.qkv_ld) = make_uint4(o[0], o[1], o[2], o[3]);
    if (units) {
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < 4; ++k) ss = fmaf(bf_lo(o[k]), bf_lo(o[k]), fmaf(bf_hi(o[k]), bf_hi(o[k]), ss));
      for (int s = 1; s < lanes; s <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
      if (live && ch < 2 * gd && g8 % lanes == 0)
        c.unit[(size_t)(t0 + i) * 2 * p.G + ch / p.D] = 1.f / sqrtf(ss + 1e-6f) / (ch < gd ? sqrtf((float)p.D) : 1.f);
    }
  };
  for (int i0 = 0; i0 < nt; i0 += PV_AHEAD) {
    uint4 in[PV_AHEAD];
#pragma unroll
    for (int a = 0; a < PV_AHEAD; ++a)
      if (i0 + a < nt) in[a] = *reinterpret_cast<const uint4*>(src + (long long)(i0 + a) * p.ld);
#pragma unroll
    for (int a = 0; a < PV_AHEAD; ++a)
      if (i0 + a < nt) token(i0 + a, in[a]);
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
  extern __shared__ float sc_s[];      // q [SC_TOK][D], k [SC_TOK][D], v [SC_TOK][32], decays [SC_TOK][D] (channel)
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
  float* gr_s = v_s + SC_TOK * 32;
  const bool channel = p.kind == REC_CHANNEL;
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
      if (rec_corrects(p.kind)) {
        rq = c.unit[(size_t)(t0 + b0 + j) * 2 * p.G + grp];
        rk = c.unit[(size_t)(t0 + b0 + j) * 2 * p.G + p.G + grp];
      }
      q_s[i] = to_f<T>(x[0]) * rq;
      k_s[i] = to_f<T>(x[gd]) * rk;
      if (channel) gr_s[i] = rec_row_decay(p, t0 + b0 + j, h, d);
    }
    for (int i = tid; i < cnt * 32; i += 256) {
      const int j = i / 32, d = i % 32;
      v_s[i] = tile0 + d < p.V ? to_f<T>(((const T*)c.qkv)[(size_t)(t0 + b0 + j) * c.qkv_ld + c.v_off + h * p.V + tile0 + d]) : 0.f;
    }
    if (tid < cnt) {
      const float* gt = c.gates + ((size_t)(t0 + b0 + tid) * p.H + h) * 2;
      g_s[tid] = p.decay ? p.decay[h] : expf(gt[0]);
      coef_s[tid] = gt[1];
    }
    __syncthreads();
    for (int j = 0; j < cnt; ++j) {
      const float g = g_s[j], v = v_s[j * 32 + warp * SC_COLS + (lane & 3)];
      float u = coef_s[j] * v;
      if (channel) {
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
          const int n = r + 8 * i;
          if (n < p.D) s[i] = fmaf(gr_s[j * p.D + n], s[i], s[i]);
        }
      }
      if (rec_corrects(p.kind)) {
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
  const int sm = SC_TOK * ((p.kind == REC_CHANNEL ? 3 : 2) * p.D + 32) * 4;
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
  if (p->kind < 0 || p->kind > 3 || (p->kind == REC_CHANNEL && (!p->step || !p->dt_bias)) || p->H < 1 || p->G < 1 || p->H % p->G != 0) return -1;
  if (p->D < 1 || p->D > REC_MAX_D || p->V < 1 || p->taps < 1 || p->H > 65535) return -1;
  if (p->taps > 1 && p->tail == nullptr) return -1;
  return 0;
}

}  // namespace skein

// Whether skein_rec_step applies a head's norm and gate too (a RecGate with out set).
extern "C" int skein_rec_step_gates(const SkeinRecParams* p) {
  using namespace skein;
  const bool pow2 = p->V >= 32 && p->V <= 256 && (p->V & (p->V - 1)) == 0;
  return pow2 && (long long)p->D * p->V * 4 <= RSB_MAX && p->D * p->V >= 2048 ? 1 : 0;
}

extern "C" int skein_rec_step(const SkeinRecParams* p, const SkeinRecGate* g, int B, int fp32, void* stream) {
  using namespace skein;
  if (B == 0) return 0;
  if (int e = rec_check(p)) return e;
  // small batches of large states: more, smaller CTAs
  const bool bulk = skein_rec_step_gates(p) && (g->out != nullptr || (long long)B * p->H >= 148);
  if (bulk) return fp32 ? rec_step_bulk<float>(*p, *g, B, (cudaStream_t)stream) : rec_step_bulk<__nv_bfloat16>(*p, *g, B, (cudaStream_t)stream);
  if (g->out != nullptr) return -1;
  return fp32 ? rec_step_any<float>(*p, B, (cudaStream_t)stream) : rec_step_any<__nv_bfloat16>(*p, B, (cudaStream_t)stream);
}

extern "C" int skein_rec_prep(const SkeinRecParams* p, const SkeinRecChunk* c, int T, int fp32, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (int e = rec_check(p)) return e;
  const int lanes = p->D / 8;
  const bool vec = !fp32 && p->D % 8 == 0 && p->V % 8 == 0 && p->ld % 8 == 0 && p->q_col % 8 == 0 && p->k_col % 8 == 0 && p->v_col % 8 == 0 &&
                   c->qkv_ld % 8 == 0 && c->v_off % 8 == 0 && p->taps <= 4 && (p->kind == REC_LIGHTNING || p->taps > 1) && (uintptr_t)p->row % 16 == 0 &&
                   (!rec_corrects(p->kind) || (lanes <= 32 && (lanes & (lanes - 1)) == 0));
  if (vec) {
    const dim3 grid(((2 * p->G * p->D + p->H * p->V) / 8 + 255) / 256 + 1, (T + PV_TOK - 1) / PV_TOK);
    auto go = [&](auto fn) -> int { return (int)launch_pdl(fn, grid, dim3(256), 0, (cudaStream_t)stream, *p, *c, T); };
    switch (p->kind == REC_LIGHTNING ? 1 : p->taps) {
      case 1: return go(rec_prep_vec_kernel<1>);
      case 2: return go(rec_prep_vec_kernel<2>);
      case 3: return go(rec_prep_vec_kernel<3>);
      default: return go(rec_prep_vec_kernel<4>);
    }
  }
  const size_t sm = rec_corrects(p->kind) ? (size_t)2 * p->G * p->D * 4 : 0;
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
  const int want = (p->C * (p->taps - 1) + 255) / 256;
  const dim3 grid(S, want < 64 ? want : 64);
  return (int)(fp32 ? launch_pdl(rec_tail_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, *p, *c)
                    : launch_pdl(rec_tail_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, *p, *c));
}
