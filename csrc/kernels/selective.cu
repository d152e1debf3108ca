// Selective scan (Mamba): a short causal convolution over time with silu, and a diagonal recurrence per channel c and state dimension n
// with a 32-bit state per sequence:
//
//   S[n, c] <- exp(dt[c] A[n, c]) S[n, c] + dt[c] u[c] B[n],    y[c] = sum_n S[n, c] C[n] + D[c] u[c],    out = y silu(z)
//
// with u the convolved channels, dt = softplus(raw + bias) and B, C projections of u that all channels share. The products that make
// B, C and raw from u run between the two kernels.
//
// A sequence owns one slot of the state pools: S [slots, N, I] fp32 and the convolution's last inputs [slots, taps, I] in the activation
// type, position p in row p mod taps (taps - 1 rows would hold the state; with one more, a decode step writes no row it reads). Position 0
// starts from zero whatever the slot holds.
//
//   short_conv   convolution and silu of every row of the step; a decode step also keeps its input
//   scan_step    decode: one row per sequence. Four channels per thread, the state read and written once
//   scan_rows    portions of sequences, one token after the other: a channel's states are spread over P lanes of a warp, tiles of tokens
//                go through shared memory while the next tile is on its way; keeps the convolution's last inputs
//
// Activations are bf16, or fp32 when a model runs in 32-bit; decays, step sizes and the state are 32-bit. Compiled without fast-math.
#include "act.cuh"
#include "launch.cuh"
#include "ptx.cuh"
#include "vec.cuh"
#include <math.h>

// Mirrored in skein_b200/ops/_lib.py (same field order).
extern "C" typedef struct SkeinScanParams {
  const void* x;             // [T, x_ld] inputs of the convolution, activation type
  void* xc;                  // [T, I] convolved: written by short_conv, read by the scan
  const void* proj;          // [T, proj_ld] B from column b_col, C from column c_col
  const float* dt;           // [T, I] step sizes before bias and softplus
  const void* z;             // [T, x_ld]
  void* out;                 // [T, out_ld]
  float* state;              // [slots, N, I]
  void* tail;                // [slots, taps, I] or null (taps == 1)
  const float* conv_w;       // [taps, I]
  const float* conv_b;       // [I]
  const float* dt_bias;      // [I]
  const float* neg_a;        // [N, I]
  const float* skip;         // [I]
  const int32_t* positions;  // [T], -1: padding row
  const int32_t* slots;      // [S]
  const int32_t* seq_of_token;   // [T], null in a decode step (row = sequence)
  const int32_t* q_start;    // [S] first row of each sequence's portion
  const int32_t* q_len;      // [S]
  int32_t* status;
  int64_t x_ld, proj_ld, out_ld;
  int32_t I, N, taps, b_col, c_col, num_slots;
} SkeinScanParams;

namespace skein {

using ScanParams = SkeinScanParams;

// ---- convolution ----------------------------------------------------------------------------------------
constexpr int SC_RUN = 8;      // consecutive rows of a thread

// V channels per thread; TAPS 0: any number. DECODE: every row is the next token of its own sequence.
template <typename T, int V, int TAPS, bool DECODE>
__global__ void __launch_bounds__(128) short_conv_kernel(const ScanParams p, int rows) {
  pdl_trigger();
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (c >= p.I) return;
  const int taps = TAPS > 0 ? TAPS : p.taps;
  const int t0 = blockIdx.y * (DECODE ? 1 : SC_RUN), t1 = min(rows, t0 + (DECODE ? 1 : SC_RUN));
  const T* x = (const T*)p.x;
  constexpr int HN = TAPS > 1 ? TAPS - 1 : 1;
  float bias[V], w[TAPS > 0 ? TAPS : 1][V], hist[HN][V];
  load_v<float, V>(p.conv_b + c, bias);
#pragma unroll
  for (int j = 0; j < TAPS; ++j) load_v<float, V>(p.conv_w + (size_t)j * p.I + c, w[j]);
  for (int t = t0; t < t1; ++t) {
    const int pos = p.positions[t];
    if (pos < 0) continue;
    const int seq = DECODE ? t : p.seq_of_token[t], first = DECODE ? t : p.q_start[seq];
    int slot = taps > 1 ? p.slots[seq] : 0;
    if (slot < 0 || slot >= p.num_slots) { report_status(p.status, ST_BAD_INDEX, slot); slot = 0; }
    // the input j tokens before row t (loaded from the row itself where there is none)
    auto prev = [&](int j, float* v) {
      const T* src = x + (size_t)t * p.x_ld + c;
      if (pos >= j) src = t - j >= first ? src - (size_t)j * p.x_ld : (const T*)p.tail + ((size_t)slot * taps + (pos - j) % taps) * p.I + c;
      load_v<T, V>(src, v);
#pragma unroll
      for (int k = 0; k < V; ++k) v[k] = pos >= j ? v[k] : 0.f;
    };
    float cur[V], a[V];
    load_v<T, V>(x + (size_t)t * p.x_ld + c, cur);
#pragma unroll
    for (int k = 0; k < V; ++k) a[k] = bias[k];
    if (TAPS > 0) {
      if (t == t0 || t == first)
#pragma unroll
        for (int j = 1; j < TAPS; ++j) prev(j, hist[j - 1]);
#pragma unroll
      for (int j = TAPS - 1; j > 0; --j)
#pragma unroll
        for (int k = 0; k < V; ++k) a[k] = fmaf(w[TAPS - 1 - j][k], hist[j - 1][k], a[k]);
#pragma unroll
      for (int k = 0; k < V; ++k) a[k] = fmaf(w[TAPS > 0 ? TAPS - 1 : 0][k], cur[k], a[k]);
    } else {
      float v[V], wj[V];
      for (int j = taps - 1; j >= 0; --j) {
        if (j > 0) prev(j, v);
        load_v<float, V>(p.conv_w + (size_t)(taps - 1 - j) * p.I + c, wj);
#pragma unroll
        for (int k = 0; k < V; ++k) a[k] = fmaf(wj[k], j > 0 ? v[k] : cur[k], a[k]);
      }
    }
    if (DECODE && taps > 1) store_v<T, V>((T*)p.tail + ((size_t)slot * taps + pos % taps) * p.I + c, cur);
#pragma unroll
    for (int k = 0; k < V; ++k) a[k] = silu_act<T>(a[k]);
    store_v<T, V>((T*)p.xc + (size_t)t * p.I + c, a);
    if (TAPS > 1) {
#pragma unroll
      for (int j = HN - 1; j > 0; --j)
#pragma unroll
        for (int k = 0; k < V; ++k) hist[j][k] = hist[j - 1][k];
#pragma unroll
      for (int k = 0; k < V; ++k) hist[0][k] = cur[k];
    }
  }
}

// exp(dt a) s + b. A decay near one is raised to a high power over a long sequence: in a 32-bit model it is taken as 1 + expm1, whose error
// shrinks with the step.
template <typename T> __device__ __forceinline__ float scan_update(float dt, float a, float s, float b);
template <> __device__ __forceinline__ float scan_update<float>(float dt, float a, float s, float b) { return fmaf(expm1f(dt * a), s, s + b); }
template <> __device__ __forceinline__ float scan_update<__nv_bfloat16>(float dt, float a, float s, float b) { return fmaf(expf(dt * a), s, b); }

// ---- decode -----------------------------------------------------------------------------------------------
constexpr int ST_THREADS = 128, ST_UNROLL = 8;

// grid (I / (128 V), B)
template <typename T, int V>
__global__ void __launch_bounds__(ST_THREADS) scan_step_kernel(const ScanParams p) {
  extern __shared__ float bc_s[];      // B [N], C [N]
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y, c = (blockIdx.x * ST_THREADS + threadIdx.x) * V, N = p.N;
  const int pos = p.positions[b];
  if (pos < 0) return;
  const int slot = p.slots[b];
  if (slot < 0 || slot >= p.num_slots) { if (threadIdx.x == 0) report_status(p.status, ST_BAD_INDEX, slot); return; }
  const bool in = c < p.I;
  float* S = p.state + (size_t)slot * N * p.I + c;
  const float* A = p.neg_a + c;
  float s[ST_UNROLL][V], an[ST_UNROLL][V];
  auto fetch = [&](int n0) {
#pragma unroll
    for (int i = 0; i < ST_UNROLL; ++i) {
#pragma unroll
      for (int k = 0; k < V; ++k) s[i][k] = an[i][k] = 0.f;
      if (in && n0 + i < N) {
        if (pos > 0) load_v<float, V>(S + (size_t)(n0 + i) * p.I, s[i]);
        load_v<float, V>(A + (size_t)(n0 + i) * p.I, an[i]);
      }
    }
  };
  fetch(0);      // the state's latency covers the rest
  const T* pr = (const T*)p.proj + (size_t)b * p.proj_ld;
  for (int i = threadIdx.x; i < 2 * N; i += ST_THREADS) bc_s[i] = to_f<T>(pr[i < N ? p.b_col + i : p.c_col + i - N]);
  float dt[V], u[V], dx[V], y[V], z[V], skip[V];
#pragma unroll
  for (int k = 0; k < V; ++k) dt[k] = u[k] = dx[k] = y[k] = z[k] = skip[k] = 0.f;
  if (in) {
    float bias[V];
    load_v<float, V>(p.dt + (size_t)b * p.I + c, dt);
    load_v<float, V>(p.dt_bias + c, bias);
    load_v<T, V>((const T*)p.xc + (size_t)b * p.I + c, u);
    load_v<T, V>((const T*)p.z + (size_t)b * p.x_ld + c, z);
    load_v<float, V>(p.skip + c, skip);
#pragma unroll
    for (int k = 0; k < V; ++k) { dt[k] = softplus_f(dt[k] + bias[k]); dx[k] = dt[k] * u[k]; y[k] = skip[k] * u[k]; }
  }
  __syncthreads();
  if (!in) return;
  for (int n0 = 0; n0 < N; n0 += ST_UNROLL) {
    if (n0 > 0) fetch(n0);
#pragma unroll
    for (int i = 0; i < ST_UNROLL; ++i) {
      if (n0 + i >= N) break;
      const float B = bc_s[n0 + i], C = bc_s[N + n0 + i];
#pragma unroll
      for (int k = 0; k < V; ++k) {
        s[i][k] = scan_update<T>(dt[k], an[i][k], s[i][k], dx[k] * B);
        y[k] = fmaf(s[i][k], C, y[k]);
      }
      store_v<float, V>(S + (size_t)(n0 + i) * p.I, s[i]);
    }
  }
#pragma unroll
  for (int k = 0; k < V; ++k) y[k] *= silu_act<T>(z[k]);
  store_v<T, V>((T*)p.out + (size_t)b * p.out_ld + c, y);
}

// ---- portions ------------------------------------------------------------------------------------------------
constexpr int SR_THREADS = 128;

// scan_update with `a` as scan_coef left it (in a bf16 model the logarithm's base is 2)
template <typename T> __device__ __forceinline__ float scan_coef(float a);
template <> __device__ __forceinline__ float scan_coef<float>(float a) { return a; }
template <> __device__ __forceinline__ float scan_coef<__nv_bfloat16>(float a) { return a * 1.44269504f; }
template <typename T> __device__ __forceinline__ float scan_size(float z);
template <> __device__ __forceinline__ float scan_size<float>(float z) { return softplus_f(z); }
template <> __device__ __forceinline__ float scan_size<__nv_bfloat16>(float z) { return softplus_series(z); }
// two of them, and two products summed, as pairs (one instruction each where the model is bf16)
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float x, float y) { f32x2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y)); return r; }
__device__ __forceinline__ float2 unpack2(f32x2 v) { float2 r; asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v)); return r; }
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) { f32x2 r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) { f32x2 r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r; }
template <typename T> __device__ __forceinline__ f32x2 scan_update2(f32x2 dt, f32x2 a, f32x2 s, f32x2 b);
template <> __device__ __forceinline__ f32x2 scan_update2<float>(f32x2 dt, f32x2 a, f32x2 s, f32x2 b) {
  const float2 d = unpack2(dt), aa = unpack2(a), ss = unpack2(s), bb = unpack2(b);
  return pack2(scan_update<float>(d.x, aa.x, ss.x, bb.x), scan_update<float>(d.y, aa.y, ss.y, bb.y));
}
template <> __device__ __forceinline__ f32x2 scan_update2<__nv_bfloat16>(f32x2 dt, f32x2 a, f32x2 s, f32x2 b) {
  const float2 x = unpack2(mul2(dt, a));
  float e0, e1;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e0) : "f"(x.x));
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e1) : "f"(x.y));
  return fma2(pack2(e0, e1), s, b);
}

// grid (I / CH, S). Lane q of a channel's P lanes holds states q RPT .. q RPT + RPT - 1; TT tokens per tile, four at a time: their decays
// do not depend on one another, and the P lanes' sums of the four outputs are formed together (a lane ends up with one token's).
template <typename T, int P, int RPT, int TT>
__global__ void __launch_bounds__(SR_THREADS, 4) scan_rows_kernel(const ScanParams p) {
  constexpr int CH = SR_THREADS / P, NP = P * RPT, EL = TT * CH / SR_THREADS, BL = (TT * NP + SR_THREADS - 1) / SR_THREADS;
  constexpr int LD = TT + 4;
  __shared__ __align__(16) float dt_s[CH][LD], dx_s[CH][LD], y_s[CH][LD];
  __shared__ __align__(16) float B_s[TT][NP], C_s[TT][NP];
  pdl_trigger();
  pdl_wait();
  const int seq = blockIdx.y, tid = threadIdx.x, c0 = blockIdx.x * CH;
  const int n_rows = p.q_len[seq];
  if (n_rows < 1) return;
  const int t0 = p.q_start[seq], pos0 = p.positions[t0];
  if (pos0 < 0) return;
  const int slot = p.slots[seq];
  if (slot < 0 || slot >= p.num_slots) { if (tid == 0) report_status(p.status, ST_BAD_INDEX, slot); return; }
  const int q = tid % P, ch = tid / P, c = c0 + ch;
  const bool in = c < p.I;
  float* S = p.state + (size_t)slot * p.N * p.I + c;
  f32x2 s[RPT / 2], a[RPT / 2];      // pairs of states
#pragma unroll
  for (int i = 0; i < RPT; i += 2) {
    float sv[2], av[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int n = q * RPT + i + k;
      const bool have = in && n < p.N;
      sv[k] = have && pos0 > 0 ? S[(size_t)n * p.I] : 0.f;
      av[k] = have ? scan_coef<T>(p.neg_a[(size_t)n * p.I + c]) : 0.f;
    }
    s[i / 2] = pack2(sv[0], sv[1]);
    a[i / 2] = pack2(av[0], av[1]);
  }
  // elements e of a tile that this thread moves: token e / CH, channel e % CH with e = tid + 128 k
  const int lc = c0 + tid % CH;
  const bool lin = lc < p.I;
  const float bias = lin ? p.dt_bias[lc] : 0.f, skip = lin ? p.skip[lc] : 0.f;
  // Loads go to clamped addresses and stay as they are until the next tile starts: all of a tile's are on their way together.
  const int lcc = lin ? lc : p.I - 1, row_max = n_rows - 1;
  float u[EL], nd[EL];
  T nu[EL], nz[EL], z[EL], nb[BL], nc[BL];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int k = 0; k < EL; ++k) {
      const size_t t = t0 + min(r0 + tid / CH + k * P, row_max);
      nu[k] = ((const T*)p.xc)[t * p.I + lcc];
      nd[k] = p.dt[t * p.I + lcc];
      nz[k] = ((const T*)p.z)[t * p.x_ld + lcc];
    }
#pragma unroll
    for (int k = 0; k < BL; ++k) {
      const int e = tid + k * SR_THREADS, n = min(e % NP, p.N - 1);
      const T* pr = (const T*)p.proj + (size_t)(t0 + min(r0 + e / NP, row_max)) * p.proj_ld;
      nb[k] = pr[p.b_col + n];
      nc[k] = pr[p.c_col + n];
    }
  };
  fetch(0);
  for (int r0 = 0; r0 < n_rows; r0 += TT) {
    const int cnt = min(TT, n_rows - r0);
#pragma unroll
    for (int k = 0; k < EL; ++k) {
      const int e = tid + k * SR_THREADS;
      u[k] = to_f<T>(nu[k]);
      z[k] = nz[k];
      const float d = r0 + e / CH < n_rows ? scan_size<T>(nd[k] + bias) : 0.f;      // a step of size zero past the end
      dt_s[e % CH][e / CH] = d;
      dx_s[e % CH][e / CH] = d * u[k];
    }
#pragma unroll
    for (int k = 0; k < BL; ++k) {
      const int e = tid + k * SR_THREADS;
      const bool have = e % NP < p.N;      // states past N take part with zeros
      if (TT * NP % SR_THREADS == 0 || e < TT * NP) {
        B_s[e / NP][e % NP] = have ? to_f<T>(nb[k]) : 0.f;
        C_s[e / NP][e % NP] = have ? to_f<T>(nc[k]) : 0.f;
      }
    }
    __syncthreads();
    if (r0 + TT < n_rows) fetch(r0 + TT);
    for (int j = 0; j < cnt; j += 4) {
      const float4 d4 = *reinterpret_cast<const float4*>(&dt_s[ch][j]), x4 = *reinterpret_cast<const float4*>(&dx_s[ch][j]);
      const float d[4] = {d4.x, d4.y, d4.z, d4.w}, x[4] = {x4.x, x4.y, x4.z, x4.w};
      float y[4];
#pragma unroll
      for (int h = 0; h < 4; ++h) {
        const f32x2 d2 = pack2(d[h], d[h]), x2 = pack2(x[h], x[h]);
        f32x2 y2 = pack2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < RPT; i += 4) {
          const ulonglong2 B = *reinterpret_cast<const ulonglong2*>(&B_s[j + h][q * RPT + i]), C = *reinterpret_cast<const ulonglong2*>(&C_s[j + h][q * RPT + i]);
          s[i / 2] = scan_update2<T>(d2, a[i / 2], s[i / 2], mul2(x2, B.x));
          s[i / 2 + 1] = scan_update2<T>(d2, a[i / 2 + 1], s[i / 2 + 1], mul2(x2, B.y));
          y2 = fma2(s[i / 2 + 1], C.y, fma2(s[i / 2], C.x, y2));
        }
        const float2 yv = unpack2(y2);
        y[h] = yv.x + yv.y;
      }
      if (P == 1) {
        *reinterpret_cast<float4*>(&y_s[ch][j]) = make_float4(y[0], y[1], y[2], y[3]);
      } else {
        const bool b0 = q & 1, b1 = q & 2;
        float v = b0 ? y[2] : y[0], w = b0 ? y[3] : y[1];
        v += __shfl_xor_sync(0xffffffffu, b0 ? y[0] : y[2], 1);
        w += __shfl_xor_sync(0xffffffffu, b0 ? y[1] : y[3], 1);
        if (P == 2) {
          *reinterpret_cast<float2*>(&y_s[ch][j + 2 * b0]) = make_float2(v, w);
        } else {
          float r = (b1 ? w : v) + __shfl_xor_sync(0xffffffffu, b1 ? v : w, 2);
#pragma unroll
          for (int o = 4; o < P; o <<= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
          if (P == 4 || q < 4) y_s[ch][j + 2 * b0 + b1] = r;
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < EL; ++k) {
      const int e = tid + k * SR_THREADS, r = r0 + e / CH;
      if (lin && r < n_rows)
        ((T*)p.out)[(size_t)(t0 + r) * p.out_ld + lc] = from_f<T>((y_s[e % CH][e / CH] + skip * u[k]) * silu_act<T>(to_f<T>(z[k])));
    }
  }
#pragma unroll
  for (int i = 0; i < RPT; i += 2) {
    const int n = q * RPT + i;
    const float2 v = unpack2(s[i / 2]);
    if (in && n < p.N) S[(size_t)n * p.I] = v.x;
    if (in && n + 1 < p.N) S[(size_t)(n + 1) * p.I] = v.y;
  }
  if (p.taps > 1) {      // every reader of the old inputs (short_conv) is done
    const int keep = min(p.taps - 1, n_rows);
    for (int e = tid; e < keep * CH; e += SR_THREADS) {
      const int r = n_rows - keep + e / CH, cc = c0 + e % CH;
      if (cc < p.I) ((T*)p.tail)[((size_t)slot * p.taps + (pos0 + r) % p.taps) * p.I + cc] = ((const T*)p.x)[(size_t)(t0 + r) * p.x_ld + cc];
    }
  }
}

template <typename T, int V, bool DECODE>
static int short_conv_go(const ScanParams& p, int rows, cudaStream_t s) {
  const dim3 grid((p.I + 128 * V - 1) / (128 * V), DECODE ? rows : (rows + SC_RUN - 1) / SC_RUN);
  auto go = [&](auto fn) -> int { return (int)launch_pdl(fn, grid, dim3(128), 0, s, p, rows); };
  switch (p.taps) {
    case 1: return go(short_conv_kernel<T, V, 1, DECODE>);
    case 2: return go(short_conv_kernel<T, V, 2, DECODE>);
    case 3: return go(short_conv_kernel<T, V, 3, DECODE>);
    case 4: return go(short_conv_kernel<T, V, 4, DECODE>);
    default: return go(short_conv_kernel<T, V, 0, DECODE>);
  }
}

template <typename T>
static int scan_rows_any(const ScanParams& p, int S, cudaStream_t s) {
  auto go = [&](auto fn, int ch) -> int { return (int)launch_pdl(fn, dim3((p.I + ch - 1) / ch, S), dim3(SR_THREADS), 0, s, p); };
  if (p.N <= 4) return go(scan_rows_kernel<T, 1, 4, 16>, 128);
  if (p.N <= 8) return go(scan_rows_kernel<T, 2, 4, 32>, 64);
  if (p.N <= 16) return go(scan_rows_kernel<T, 4, 4, 32>, 32);
  if (p.N <= 32) return go(scan_rows_kernel<T, 8, 4, 32>, 16);
  if (p.N <= 64) return go(scan_rows_kernel<T, 16, 4, 32>, 8);
  if (p.N <= 128) return go(scan_rows_kernel<T, 16, 8, 16>, 8);
  if (p.N <= 256) return go(scan_rows_kernel<T, 16, 16, 16>, 8);
  return -1;
}

static int scan_check(const ScanParams* p) {
  if (p->I < 1 || p->N < 1 || p->taps < 1 || (p->taps > 1 && p->tail == nullptr)) return -1;
  return 0;
}
// 4-element accesses to rows of x, z, xc, out and the state
static bool scan_vec(const ScanParams* p) {
  auto ok = [](const void* q) { return (uintptr_t)q % 16 == 0; };
  return p->I % 4 == 0 && p->x_ld % 4 == 0 && p->out_ld % 4 == 0 && ok(p->x) && ok(p->z) && ok(p->out) && ok(p->xc) && ok(p->dt) && ok(p->tail) && ok(p->state);
}

}  // namespace skein

extern "C" int skein_short_conv(const SkeinScanParams* p, int rows, int decode, int fp32, void* stream) {
  using namespace skein;
  if (rows == 0) return 0;
  if (int e = scan_check(p)) return e;
  cudaStream_t s = (cudaStream_t)stream;
  const bool v = scan_vec(p);
  if (fp32) {
    if (decode) return v ? short_conv_go<float, 4, true>(*p, rows, s) : short_conv_go<float, 1, true>(*p, rows, s);
    return v ? short_conv_go<float, 4, false>(*p, rows, s) : short_conv_go<float, 1, false>(*p, rows, s);
  }
  if (decode) return v ? short_conv_go<__nv_bfloat16, 4, true>(*p, rows, s) : short_conv_go<__nv_bfloat16, 1, true>(*p, rows, s);
  return v ? short_conv_go<__nv_bfloat16, 4, false>(*p, rows, s) : short_conv_go<__nv_bfloat16, 1, false>(*p, rows, s);
}

extern "C" int skein_scan_step(const SkeinScanParams* p, int B, int fp32, void* stream) {
  using namespace skein;
  if (B == 0) return 0;
  if (int e = scan_check(p)) return e;
  if (p->N > 4096) return -1;
  const int v = scan_vec(p) ? 4 : 1;
  const dim3 grid((p->I + ST_THREADS * v - 1) / (ST_THREADS * v), B);
  auto go = [&](auto fn) -> int { return (int)launch_pdl(fn, grid, dim3(ST_THREADS), (size_t)p->N * 8, (cudaStream_t)stream, *p); };
  if (fp32) return v == 4 ? go(scan_step_kernel<float, 4>) : go(scan_step_kernel<float, 1>);
  return v == 4 ? go(scan_step_kernel<__nv_bfloat16, 4>) : go(scan_step_kernel<__nv_bfloat16, 1>);
}

// State dimensions up to 256.
extern "C" int skein_scan_rows(const SkeinScanParams* p, int S, int fp32, void* stream) {
  using namespace skein;
  if (S == 0) return 0;
  if (int e = scan_check(p)) return e;
  return fp32 ? scan_rows_any<float>(*p, S, (cudaStream_t)stream) : scan_rows_any<__nv_bfloat16>(*p, S, (cudaStream_t)stream);
}
