// The delta rule with a decay per row of the state (recurrent.cu: channel) over whole chunks of 64 tokens on the tensor cores (bf16 models,
// D = 64 or 128, V a multiple of 64). With G_i [D] the running sums of the log decays inside a chunk, S the state before it, q and k unit
// vectors (q times D^-1/2), all products of two vectors element by element:
//
//   U   = T diag(beta) (V - K+ S)                        K+_i = k_i e^G_i
//   O   = Q+ S + P U                                     Q+_i = q_i e^G_i,   P_ij = q_i . (k_j e^(G_i - G_j)), j <= i
//   S  <- e^G_last S + K-^T U                            K-_i = k_i e^(G_last - G_i)
//   T   = (I + A)^-1,   A_ij = beta_i k_i . (k_j e^(G_i - G_j)), j < i
//
//   rec_channel_mats   every chunk and head at once: T (hi + lo), P, K+ and K- (hi + lo), Q+, beta, e^G_last
//   rec_channel_chunk  one CTA per (128 columns of V, head, sequence) walks the chunks, everything transposed as in recurrent_tc.cu:
//                          warp 0      TMA                     warp 1   MMA issue (one lane)
//                          warps 2-9   two threads per column of V: half of the state's rows (fp32 registers) and half of the tokens each
//                      V and the matrices are two chunks ahead; K+ and Q+ are read by a chunk's first product and K- by its last, so
//                      that one buffer each is filled again in time
//
// e^(G_i - G_j) does not split into a factor of the row and one of the column that both stay in range: decays can be arbitrarily strong. The
// chunk's 16 x 16 blocks below the diagonal take e^(G_i - G_ref) and e^(G_ref - G_j) with the reference at the start of block i, both at most
// one. A block on the diagonal does the same where its decays allow it (e^(G_ref - G_j) at most e^60), else it sums element by element.
// Sums of logarithms run inside blocks of 16 tokens only, so that their differences keep the accuracy of 32-bit.
//
// The state is fp32 from chunk to chunk; as an operand it and whatever flows back into it (K+, K-, U, T) are two bf16 summands. The read-out
// takes Q+, P and U in bf16. Every wait is bounded. Compiled without fast-math.
#include "act.cuh"
#include "ptx.cuh"
#include "launch.cuh"
#include "recurrent.cuh"
#include "recurrent_tc.cuh"
#include <cuda.h>
#include <cuda_bf16.h>
#include <math.h>

namespace skein {

int cached_tmap_2d(CUtensorMap* out, const void* base, uint64_t rows, uint64_t k_elems, int elem_bytes, uint32_t box_rows);

constexpr int RC_NOPS = 5;                 // operand matrices [64][D] of a chunk: K+ hi, Q+, K+ lo, K- hi, K- lo
constexpr int RC_B = 16;                   // tokens of a block
constexpr float RC_MAX_LOG2 = 86.f;        // a block whose decays sum up to less (base 2) takes the factored form
__host__ __device__ constexpr int rc_factors(int d) { return RT_C + d; }      // floats of a chunk: beta, e^G_last

__device__ __forceinline__ float rc_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// ---- the chunks' matrices ---------------------------------------------------------------------------
// column operands [64][D + 8] hi, lo (T's and the inverse's scratch take their place later), row operands K, Q [16][D + 8] hi, lo, A, running
// sums [64][D], sums of the blocks [4][D]
__host__ __device__ constexpr int rc_mats_smem(int d) {
  return 2 * RT_C * (d + 8) * 2 + 4 * RC_B * (d + 8) * 2 + 2 * RT_C * RT_LX * 2 + RT_C * RT_LD * 4 + RT_C * d * 4 + 4 * d * 4;
}

__device__ __forceinline__ void rc_unpack8(const uint4& u, float* v) {
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) { v[2 * i] = __uint_as_float(w[i] << 16); v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u); }
}
__device__ __forceinline__ void rc_split8(const float* v, uint4& hi, uint4& lo) {
  rt_split(v[0], v[1], hi.x, lo.x);
  rt_split(v[2], v[3], hi.y, lo.y);
  rt_split(v[4], v[5], hi.z, lo.z);
  rt_split(v[6], v[7], hi.w, lo.w);
}
__device__ __forceinline__ void rc_load8(const float* p, float* v) {
  *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
  *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(p + 4);
}

// grid (chunks, H, S), 256 threads
template <int D>
__global__ void __launch_bounds__(256, 2) rec_channel_mats_kernel(const RecParams p, const RecChunk c, __nv_bfloat16* mats, __nv_bfloat16* opers,
                                                                  float* factors) {
  extern __shared__ __align__(16) uint8_t mt_smem[];
  __shared__ float beta_s[RT_C], rq_s[RT_C], rk_s[RT_C];
  __shared__ int strong_s;                 // bit b: block b's decays are too strong for the factored form
  constexpr int LD = D + 8, TPR = D / 8;   // threads of a row
  __nv_bfloat16* Ch = reinterpret_cast<__nv_bfloat16*>(mt_smem);
  __nv_bfloat16* Cl = Ch + RT_C * LD;
  __nv_bfloat16* Xh = Ch;                  // once the column operands are done with
  __nv_bfloat16* Xl = Xh + RT_C * RT_LX;
  __nv_bfloat16* Yh = Xl + RT_C * RT_LX;
  __nv_bfloat16* Yl = Yh + 32 * RT_LY;
  __nv_bfloat16* Rk = Cl + RT_C * LD;      // [K hi | K lo | Q hi | Q lo][16][LD]
  __nv_bfloat16* Ah = Rk + 4 * RC_B * LD;
  __nv_bfloat16* Al = Ah + RT_C * RT_LX;
  float* Ad = reinterpret_cast<float*>(Al + RT_C * RT_LX);
  float* L = Ad + RT_C * RT_LD;            // [64][D] running sums inside the blocks, base 2
  float* Tot = L + RT_C * D;               // [4][D]
  static_assert(2 * RT_C * RT_LX + 2 * 32 * RT_LY <= 2 * RT_C * LD + 4 * RC_B * LD, "the inverse's scratch fits the operands' place");
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.y, seq = blockIdx.z, len = c.q_len[seq], i0 = blockIdx.x * RT_C;
  if (i0 >= len) return;
  const int n = min(RT_C, len - i0), q_start = c.q_start[seq], t0 = q_start + i0;
  const int unit = (rt_chunk0(q_start, seq) + blockIdx.x) * p.H + h;
  const int grp = h / (p.H / p.G), gd = p.G * D, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) strong_s = 0;
  if (tid < RT_C) {
    const int t = t0 + (tid < n ? tid : 0);
    const float* un = c.unit + (size_t)t * 2 * p.G;
    beta_s[tid] = tid < n ? c.gates[((size_t)t * p.H + h) * 2 + 1] : 0.f;
    rq_s[tid] = un[grp];
    rk_s[tid] = un[p.G + grp];
  }
  __syncthreads();
  {      // a thread per channel and block (or two blocks): running sums of the log decays
    const int d = tid % D;
    const float nd = p.neg_decay[h] * 1.4426950408889634f, bias = p.dt_bias[h * D + d];
    for (int b = tid / D; b < 4; b += 256 / D) {
      float a[RC_B], sum = 0.f;
#pragma unroll
      for (int i = 0; i < RC_B; ++i) a[i] = b * RC_B + i < n ? p.step[(size_t)(t0 + b * RC_B + i) * p.H * D + h * D + d] : 0.f;
#pragma unroll
      for (int i = 0; i < RC_B; ++i) {
        if (b * RC_B + i < n) sum = fmaf(nd, softplus_series(a[i] + bias), sum);
        L[(b * RC_B + i) * D + d] = sum;
      }
      Tot[b * D + d] = sum;
      if (sum < -RC_MAX_LOG2) atomicOr(&strong_s, 1 << b);
    }
  }
  __syncthreads();
  const int strong = strong_s;
  const __nv_bfloat16* qkv = (const __nv_bfloat16*)c.qkv + (size_t)t0 * c.qkv_ld + grp * D;
  auto load_k = [&](int t, int col, float* v) {      // a unit key's 8 elements; zero past the portion
    uint4 u = make_uint4(0, 0, 0, 0);
    if (t < n) u = *reinterpret_cast<const uint4*>(qkv + (size_t)t * c.qkv_ld + gd + col);
    rc_unpack8(u, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= rk_s[t];
  };
  __nv_bfloat16* ops = opers + (size_t)unit * RC_NOPS * RT_C * D;
  __nv_bfloat16* out = mats + (size_t)unit * 3 * RT_C * RT_C;
  for (int b = 0; b < 4; ++b) {
    if (b > 0) __syncthreads();            // the previous block's operands have been read
    // row operands of block b, and the chunk's K+, Q+, K-
    for (int it = tid; it < RC_B * TPR; it += 256) {
      const int r = it / TPR, col = it % TPR * 8, t = b * RC_B + r;
      float k[8], q[8], l[8], x[8], before[8], after[8];
      load_k(t, col, k);
      uint4 u = make_uint4(0, 0, 0, 0);
      if (t < n) u = *reinterpret_cast<const uint4*>(qkv + (size_t)t * c.qkv_ld + col);
      rc_unpack8(u, q);
      rc_load8(L + t * D + col, l);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        q[i] *= rq_s[t];
        before[i] = l[i];
        after[i] = Tot[b * D + col + i] - l[i];
      }
      for (int o = 0; o < 4; ++o)
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float tot = o == b ? 0.f : Tot[o * D + col + i];
          if (o < b) before[i] += tot; else after[i] += tot;
        }
      uint4 hi, lo;
#pragma unroll
      for (int i = 0; i < 8; ++i) x[i] = k[i] * rc_exp2(after[i]);
      rc_split8(x, hi, lo);
      *reinterpret_cast<uint4*>(ops + (size_t)(3 * RT_C + t) * D + col) = hi;
      *reinterpret_cast<uint4*>(ops + (size_t)(4 * RT_C + t) * D + col) = lo;
#pragma unroll
      for (int i = 0; i < 8; ++i) { before[i] = rc_exp2(before[i]); x[i] = k[i] * before[i]; }
      rc_split8(x, hi, lo);
      *reinterpret_cast<uint4*>(ops + (size_t)t * D + col) = hi;
      *reinterpret_cast<uint4*>(ops + (size_t)(2 * RT_C + t) * D + col) = lo;
#pragma unroll
      for (int i = 0; i < 8; ++i) x[i] = q[i] * before[i];
      rc_split8(x, hi, lo);
      *reinterpret_cast<uint4*>(ops + (size_t)(RT_C + t) * D + col) = hi;
#pragma unroll
      for (int i = 0; i < 8; ++i) { l[i] = rc_exp2(l[i]); x[i] = k[i] * l[i]; }
      rc_split8(x, hi, lo);
      *reinterpret_cast<uint4*>(Rk + r * LD + col) = hi;
      *reinterpret_cast<uint4*>(Rk + (RC_B + r) * LD + col) = lo;
#pragma unroll
      for (int i = 0; i < 8; ++i) x[i] = q[i] * l[i];
      rc_split8(x, hi, lo);
      *reinterpret_cast<uint4*>(Rk + (2 * RC_B + r) * LD + col) = hi;
      *reinterpret_cast<uint4*>(Rk + (3 * RC_B + r) * LD + col) = lo;
    }
    // column operands: decays from the token to the start of block b (inside block b: from its start back to the token)
    const bool direct = (strong >> b) & 1;
    const int rows = (direct ? b : b + 1) * RC_B;
    for (int it = tid; it < rows * TPR; it += 256) {
      const int t = it / TPR, col = it % TPR * 8, bt = t / RC_B;
      float k[8], l[8];
      load_k(t, col, k);
      rc_load8(L + t * D + col, l);
#pragma unroll
      for (int i = 0; i < 8; ++i) l[i] = bt == b ? -l[i] : Tot[bt * D + col + i] - l[i];
      for (int o = bt + 1; o < b; ++o)
#pragma unroll
        for (int i = 0; i < 8; ++i) l[i] += Tot[o * D + col + i];
#pragma unroll
      for (int i = 0; i < 8; ++i) k[i] *= rc_exp2(l[i]);
      uint4 hi, lo;
      rc_split8(k, hi, lo);
      *reinterpret_cast<uint4*>(Ch + t * LD + col) = hi;
      *reinterpret_cast<uint4*>(Cl + t * LD + col) = lo;
    }
    __syncthreads();
    // a warp per 16 x 16 block of A (warps 0-3) and P (warps 4-7)
    const int cb = warp & 3;
    const bool qk = warp >= 4;
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    if (cb < b || (cb == b && !direct)) {
      const uint32_t ra = smem_u32(Rk + (qk ? 2 : 0) * RC_B * LD), ca = smem_u32(Ch + cb * RC_B * LD);
      constexpr uint32_t R_LO = RC_B * LD * 2, C_LO = RT_C * LD * 2;
      const int mat = lane >> 3;
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        const uint32_t a = ra + ((lane & 15) * LD + ks * 16 + (lane >> 4) * 8) * 2, x = ca + (((mat >> 1) * 8 + (lane & 7)) * LD + ks * 16 + (mat & 1) * 8) * 2;
        rt_ldsm4(a, ah);
        rt_ldsm4(a + R_LO, al);
        rt_ldsm4(x, bh);
        rt_ldsm4(x + C_LO, bl);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          rt_mma(acc[j], ah, bh[2 * j], bh[2 * j + 1]);
          rt_mma(acc[j], al, bh[2 * j], bh[2 * j + 1]);
          rt_mma(acc[j], ah, bl[2 * j], bl[2 * j + 1]);
        }
      }
    } else if (cb == b) {
      // strong decays: this lane's eight sums one element after the other
      for (int j = 0; j < 2; ++j)
        for (int e = 0; e < 4; ++e) {
          const int i = b * RC_B + (lane >> 2) + 8 * (e >> 1), s = b * RC_B + j * 8 + (lane & 3) * 2 + (e & 1);
          if (s > i || i >= n) continue;
          float sum = 0.f;
          for (int d = 0; d < D; ++d) {
            const float x = __bfloat162float(qkv[(size_t)i * c.qkv_ld + (qk ? 0 : gd) + d]), k = __bfloat162float(qkv[(size_t)s * c.qkv_ld + gd + d]);
            sum = fmaf(x * k, rc_exp2(L[i * D + d] - L[s * D + d]), sum);
          }
          acc[j][e] = sum * (qk ? rq_s[i] : rk_s[i]) * rk_s[s];
        }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int r = (lane >> 2) + 8 * hf, i = b * RC_B + r, q = j * 8 + (lane & 3) * 2, s = cb * RC_B + q;
        const int last = qk ? i : i - 1;
        float v0 = cb <= b && s <= last ? acc[j][2 * hf] : 0.f, v1 = cb <= b && s + 1 <= last ? acc[j][2 * hf + 1] : 0.f;
        if (qk) {
          *reinterpret_cast<uint32_t*>(out + 2 * RT_C * RT_C + i * RT_C + s) = rt_pack(v0, v1);
          continue;
        }
        v0 *= beta_s[i];
        v1 *= beta_s[i];
        if (cb == b) {
          Ad[i * RT_LD + q] = v0;
          Ad[i * RT_LD + q + 1] = v1;
        } else if (cb < b) {
          uint32_t hi, lo;
          rt_split(v0, v1, hi, lo);
          *reinterpret_cast<uint32_t*>(Ah + i * RT_LX + s) = hi;
          *reinterpret_cast<uint32_t*>(Al + i * RT_LX + s) = lo;
        }
      }
  }
  float* f = factors + (size_t)unit * rc_factors(D);
  if (tid < RT_C) f[tid] = beta_s[tid];
  else if (tid < RT_C + D) { const int d = tid - RT_C; f[tid] = rc_exp2(Tot[d] + Tot[D + d] + Tot[2 * D + d] + Tot[3 * D + d]); }
  __syncthreads();
  rt_invert(Ad, Ah, Xh, Xl, Yh, Yl);
  for (int i = tid; i < 2 * RT_C * 8; i += 256) {
    const int m = i / (RT_C * 8), r = i % (RT_C * 8) / 8, ch = i % 8;
    reinterpret_cast<uint4*>(out)[i] = *reinterpret_cast<const uint4*>((m ? Xl : Xh) + r * RT_LX + ch * 8);
  }
}

// ---- the walk over the chunks -------------------------------------------------------------------------
constexpr int RC_THREADS = 320, RC_COMPUTE = 256;
__host__ __device__ constexpr int rc_half_bytes() { return RT_C * 128; }                                     // 64 rows of 64 elements
__host__ __device__ constexpr int rc_stage_bytes() { return 2 * RT_C * 128 + 3 * RT_MAT_BYTES + 1024; }       // V, T hi, T lo, P, factors
__host__ __device__ constexpr int rc_first_bytes(int d) { return d / 64 * 3 * RT_C * 128; }                   // per half [K+ hi | Q+], then K+ lo
__host__ __device__ constexpr int rc_last_bytes(int d) { return d / 64 * 2 * RT_C * 128; }                    // K- hi, then K- lo
constexpr int RC_OUT_BYTES = RT_C * 256;      // a chunk's outputs, [64][128] bf16
__host__ __device__ constexpr int rc_smem(int d) { return 2 * (rc_stage_bytes() + RC_OUT_BYTES) + rc_first_bytes(d) + rc_last_bytes(d) + 1024 + 256; }

// tensor-memory columns: A operands S (hi, lo); accumulators [R | O1] of one product, U, O2, dS
constexpr uint32_t RC_SH = 0, RC_SL = 64, RC_R = 128, RC_O1 = 192, RC_U = 256, RC_O2 = 320, RC_DS = 384;

template <int D>
__global__ void __launch_bounds__(RC_THREADS, 1)
rec_channel_chunk_kernel(const __grid_constant__ CUtensorMap tmX, const __grid_constant__ CUtensorMap tmM, const __grid_constant__ CUtensorMap tmK,
                         const RecParams p, const RecChunk c, const float* factors) {
  constexpr int HALVES = D / 64, HB = rc_half_bytes(), STAGE = rc_stage_bytes();
  constexpr int OFF_M = 2 * RT_C * 128, OFF_F = OFF_M + 3 * RT_MAT_BYTES;
  const int h = blockIdx.y, seq = blockIdx.z, tile0 = blockIdx.x * 128;
  const int len = c.q_len[seq], slot = p.slots[seq];
  if (len < 1 || slot < 0 || slot >= p.num_slots) return;
  const int t0 = c.q_start[seq], n_chunks = (len + RT_C - 1) / RT_C, unit0 = rt_chunk0(t0, seq);

  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
  const uint32_t first_s = base + 2 * (STAGE + RC_OUT_BYTES), last_s = first_s + rc_first_bytes(D), bars = last_s + rc_last_bytes(D);
  const uint32_t klo_s = first_s + HALVES * 2 * HB;
  const uint32_t bar_full = bars, bar_empty = bars + 16, bar_s = bars + 32, bar_r = bars + 40, bar_rr = bars + 48, bar_u = bars + 56,
                 bar_ur = bars + 64, bar_o = bars + 72, bar_first = bars + 80, bar_last = bars + 88;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(base_ptr + (bars - base) + 96);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(base_ptr + (bars - base) + 104);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    for (int s = 0; s < 2; ++s) { mbar_init(bar_full + 8 * s, 1); mbar_init(bar_empty + 8 * s, RC_COMPUTE); }
    mbar_init(bar_s, RC_COMPUTE); mbar_init(bar_r, 1); mbar_init(bar_rr, RC_COMPUTE); mbar_init(bar_u, 1); mbar_init(bar_ur, RC_COMPUTE);
    mbar_init(bar_o, 1); mbar_init(bar_first, 1); mbar_init(bar_last, 1);
    abort_flag[0] = 0;
    abort_flag[1] = 0;      // never set: the drain waits of a failing producer run out on their time budget only
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), 512);
    tmem_relinquish();
  }
  pdl_trigger();
  pdl_wait();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tm = *tmem_slot;
  const int v_halves = min(2, (p.V - tile0 + 63) / 64);

  if (warp == 0) {
    // ---------------------------------------------------------------- TMA producer
    if (lane == 0) {
      tma_prefetch_desc(&tmX);
      tma_prefetch_desc(&tmM);
      tma_prefetch_desc(&tmK);
      const uint64_t pol = l2_policy_evict_first();
      bool ok = true;
      int armed[2] = {0, 0}, armed_first = 0, armed_last = 0;
      for (int j = 0; j < n_chunks; ++j) {
        const int s = j & 1, unit = (unit0 + j) * p.H + h;
        if (j >= 2 && !mbar_wait(bar_empty + 8 * s, ((j >> 1) - 1) & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
        const uint32_t st = base + s * STAGE, full = bar_full + 8 * s;
        mbar_expect_tx(full, v_halves * HB + 3 * RT_MAT_BYTES + rc_factors(D) * 4);
        ++armed[s];
        for (int hf = 0; hf < v_halves; ++hf) tma_load_2d(st + hf * HB, &tmX, full, c.v_off + h * p.V + tile0 + hf * 64, t0 + j * RT_C, pol);
        for (int m = 0; m < 3; ++m) tma_load_2d(st + OFF_M + m * RT_MAT_BYTES, &tmM, full, 0, (unit * 3 + m) * RT_C, pol);
        bulk_load_1d(st + OFF_F, factors + (size_t)unit * rc_factors(D), rc_factors(D) * 4, full);
        // the previous chunk's first product is complete
        if (j > 0 && !mbar_wait(bar_r, (j - 1) & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
        mbar_expect_tx(bar_first, rc_first_bytes(D));
        ++armed_first;
        const int row = unit * RC_NOPS * RT_C;
        for (int hf = 0; hf < HALVES; ++hf) {
          tma_load_2d(first_s + hf * 2 * HB, &tmK, bar_first, hf * 64, row, pol);
          tma_load_2d(first_s + hf * 2 * HB + HB, &tmK, bar_first, hf * 64, row + RT_C, pol);
          tma_load_2d(klo_s + hf * HB, &tmK, bar_first, hf * 64, row + 2 * RT_C, pol);
        }
        // ... and its last
        if (j > 0 && !mbar_wait(bar_o, (j - 1) & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
        mbar_expect_tx(bar_last, rc_last_bytes(D));
        ++armed_last;
        for (int hf = 0; hf < HALVES; ++hf)
          for (int m = 0; m < 2; ++m) tma_load_2d(last_s + (m * HALVES + hf) * HB, &tmK, bar_last, hf * 64, row + (3 + m) * RT_C, pol);
      }
      if (!ok) {
        if (*abort_flag == 0) { *abort_flag = 1; report_status(p.status, ST_TIMEOUT_SMEM_EMPTY, 40); }
        // copies already issued still write this CTA's shared memory: wait for them (bounded) before leaving
        for (int s = 0; s < 2; ++s)
          if (armed[s] > 0) mbar_wait(bar_full + 8 * s, (armed[s] - 1) & 1, abort_flag + 1, RT_BUDGET_NS);
        if (armed_first > 0) mbar_wait(bar_first, (armed_first - 1) & 1, abort_flag + 1, RT_BUDGET_NS);
        if (armed_last > 0) mbar_wait(bar_last, (armed_last - 1) & 1, abort_flag + 1, RT_BUDGET_NS);
      }
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      const uint32_t id_c = umma_idesc(1, 1, 128, RT_C), id_2c = umma_idesc(1, 1, 128, 2 * RT_C);
      const uint32_t id_d = umma_idesc(1, 1, 128, D) | (1u << 16);      // B operand MN-major
      bool ok = true;
      for (int j = 0; j < n_chunks && ok; ++j) {
        const int s = j & 1;
        const uint32_t st = base + s * STAGE;
        ok = mbar_wait(bar_first, j & 1, abort_flag, RT_BUDGET_NS) && mbar_wait(bar_s, j & 1, abort_flag, RT_BUDGET_NS);
        if (!ok) break;
        tc_fence_after();
        // [R | O1] = S [K+ | Q+]^T, then what K+ lo adds to R
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int k = 0; k < D / 16; ++k)
            mma_f16_ts(tm + RC_R, tm + (part ? RC_SL : RC_SH) + k * 8, umma_desc_sw128(first_s + (k >> 2) * 2 * HB + (k & 3) * 32), id_2c,
                       part > 0 || k > 0 ? 1u : 0u);
#pragma unroll
        for (int k = 0; k < D / 16; ++k) mma_f16_ts(tm + RC_R, tm + RC_SH + k * 8, umma_desc_sw128(klo_s + (k >> 2) * HB + (k & 3) * 32), id_c, 1u);
        tc_commit(bar_r);
        ok = mbar_wait(bar_full + 8 * s, (j >> 1) & 1, abort_flag, RT_BUDGET_NS) && mbar_wait(bar_rr, j & 1, abort_flag, RT_BUDGET_NS);
        if (!ok) break;
        tc_fence_after();
        // U = R T^T; R (hi, lo) lies where O2 will go
#pragma unroll
        for (int part = 0; part < 3; ++part)
#pragma unroll
          for (int k = 0; k < RT_C / 16; ++k)
            mma_f16_ts(tm + RC_U, tm + RC_O2 + (part == 1 ? 32 : 0) + k * 8, umma_desc_sw128(st + OFF_M + (part == 2 ? RT_MAT_BYTES : 0) + k * 32), id_c,
                       part > 0 || k > 0 ? 1u : 0u);
        tc_commit(bar_u);
        ok = mbar_wait(bar_ur, j & 1, abort_flag, RT_BUDGET_NS) && mbar_wait(bar_last, j & 1, abort_flag, RT_BUDGET_NS);
        if (!ok) break;
        tc_fence_after();
        // O2 = U P^T, dS = U K-. Operands: U (bf16) in R's columns, U (hi, lo) in S's
#pragma unroll
        for (int k = 0; k < RT_C / 16; ++k)
          mma_f16_ts(tm + RC_O2, tm + RC_R + k * 8, umma_desc_sw128(st + OFF_M + 2 * RT_MAT_BYTES + k * 32), id_c, k > 0 ? 1u : 0u);
#pragma unroll
        for (int part = 0; part < 3; ++part)
#pragma unroll
          for (int k = 0; k < RT_C / 16; ++k)
            mma_f16_ts(tm + RC_DS, tm + RC_SH + (part == 1 ? 32 : 0) + k * 8,
                       umma_desc_sw128_mn(last_s + (part == 2 ? HALVES * HB : 0) + k * 16 * 128, HB), id_d, part > 0 || k > 0 ? 1u : 0u);
        tc_commit(bar_o);
      }
      if (!ok && *abort_flag == 0) { *abort_flag = 1; report_status(p.status, ST_TIMEOUT_SMEM_FULL, 41); }
    }
  } else {
    // ---------------------------------------------------------------- state, splits, outputs: thread <-> column of V, half hf
    const int quarter = warp & 3, hf = (warp - 2) >> 2, v = quarter * 32 + lane, col = tile0 + v;
    const uint32_t ta = tm + ((uint32_t)(quarter * 32) << 16);
    const bool in = col < p.V;
    constexpr int NS = D / 2;               // rows of the state in this thread
    float* S = p.state + ((size_t)slot * p.H + h) * D * p.V + (size_t)hf * NS * p.V + col;
    const bool fresh = p.positions[t0] == 0;
    float s[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) s[i] = (in && !fresh) ? S[(size_t)i * p.V] : 0.f;
    auto put_state = [&]() {                // S as an operand, hi and lo
#pragma unroll
      for (int b = 0; b < NS / 32; ++b) {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) rt_split(s[b * 32 + 2 * i], s[b * 32 + 2 * i + 1], hi[i], lo[i]);
        tmem_st16(ta + RC_SH + hf * (NS / 2) + b * 16, hi);
        tmem_st16(ta + RC_SL + hf * (NS / 2) + b * 16, lo);
      }
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(bar_s);
    };
    const uint32_t v_byte = (uint32_t)(v & 63) * 2, v_half = (v >> 6) * HB;
    const int cols = min(128, p.V - tile0), ct = tid - 64;      // columns of the tile; number of this thread among the 256
    // V[token i][col] of a stage; 128-byte rows, 16-byte pieces swizzled by the row
    auto value = [&](int sg, int i) {
      return __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(base_ptr + sg * STAGE + v_half + i * 128 + (v_byte ^ ((i & 7) << 4))));
    };
    bool ok = true;
    put_state();
    for (int j = 0; j < n_chunks; ++j) {
      const int sg = j & 1, n = min(RT_C, len - j * RT_C);
      const float* f = reinterpret_cast<const float*>(base_ptr + sg * STAGE + OFF_F);
      if (!mbar_wait(bar_full + 8 * sg, (j >> 1) & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
      uint32_t r[32], hi[16], lo[16];
      float x[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) x[i] = in ? value(sg, hf * 32 + i) : 0.f;       // (while the product runs)
      if (!mbar_wait(bar_r, j & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
      tc_fence_after();
      tmem_ld32(ta + RC_R + hf * 32, r);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const float2 b2 = *reinterpret_cast<const float2*>(f + hf * 32 + 2 * i);
        rt_split(b2.x * (x[2 * i] - __uint_as_float(r[2 * i])), b2.y * (x[2 * i + 1] - __uint_as_float(r[2 * i + 1])), hi[i], lo[i]);
      }
      tmem_st16(ta + RC_O2 + hf * 16, hi);
      tmem_st16(ta + RC_O2 + 32 + hf * 16, lo);
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(bar_rr);
      if (!mbar_wait(bar_u, j & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
      tc_fence_after();
      tmem_ld32(ta + RC_U + hf * 32, r);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 16; ++i) rt_split(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1]), hi[i], lo[i]);
      tmem_st16(ta + RC_R + hf * 16, hi);
      tmem_st16(ta + RC_SH + hf * 16, hi);
      tmem_st16(ta + RC_SH + 32 + hf * 16, lo);
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(bar_ur);
      if (!mbar_wait(bar_o, j & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
      tc_fence_after();
      uint32_t o[16];                       // the chunk's outputs of this thread, pairs of tokens
      {
        uint32_t o1[32], o2[32];
        tmem_ld32(ta + RC_O1 + hf * 32, o1);
        tmem_ld32(ta + RC_O2 + hf * 32, o2);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i)
          o[i] = rt_pack(__uint_as_float(o1[2 * i]) + __uint_as_float(o2[2 * i]), __uint_as_float(o1[2 * i + 1]) + __uint_as_float(o2[2 * i + 1]));
      }
#pragma unroll
      for (int b = 0; b < NS / 32; ++b) {
        uint32_t d[32];
        tmem_ld32(ta + RC_DS + hf * NS + b * 32, d);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          const float4 g = *reinterpret_cast<const float4*>(f + RT_C + hf * NS + b * 32 + i);
          float* q = s + b * 32 + i;
          q[0] = fmaf(g.x, q[0], __uint_as_float(d[i])); q[1] = fmaf(g.y, q[1], __uint_as_float(d[i + 1]));
          q[2] = fmaf(g.z, q[2], __uint_as_float(d[i + 2])); q[3] = fmaf(g.w, q[3], __uint_as_float(d[i + 3]));
        }
      }
      tc_fence_before();
      mbar_arrive(bar_empty + 8 * sg);
      if (j + 1 < n_chunks) put_state();
      // the outputs go through shared memory to whole 16-byte pieces of the rows, while the next chunk's product runs. Two buffers:
      // a thread can be one chunk ahead of another here, not two.
      uint8_t* ob = base_ptr + 2 * STAGE + (j & 1) * RC_OUT_BYTES;
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        *reinterpret_cast<uint16_t*>(ob + (hf * 32 + 2 * i) * 256 + v * 2) = (uint16_t)o[i];
        *reinterpret_cast<uint16_t*>(ob + (hf * 32 + 2 * i + 1) * 256 + v * 2) = (uint16_t)(o[i] >> 16);
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");
      __nv_bfloat16* out = (__nv_bfloat16*)p.out + (size_t)(t0 + j * RT_C) * p.H * p.V + (size_t)h * p.V + tile0;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = (ct >> 4) + 16 * i, ch = ct & 15;
        if (t < n && ch * 8 < cols) *reinterpret_cast<uint4*>(out + (size_t)t * p.H * p.V + ch * 8) = *reinterpret_cast<const uint4*>(ob + t * 256 + ch * 16);
      }
    }
    if (ok) {
#pragma unroll
      for (int i = 0; i < NS; ++i)
        if (in) S[(size_t)i * p.V] = s[i];
    } else if (*abort_flag == 0) {
      *abort_flag = 1;
      report_status(p.status, ST_TIMEOUT_TMEM_FULL, 42);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tm, 512);
  }
}

static long long rc_units(const RecParams& p, int T, int S) { return (long long)(T / RT_C + S + 1) * p.H; }

template <int D>
static int rec_channel_go(const RecParams& p, const RecChunk& c, int T, int S, cudaStream_t s) {
  const long long units = rc_units(p, T, S);
  if (units * RC_NOPS * RT_C > 0x7fffffff) return -1;
  __nv_bfloat16* mats = (__nv_bfloat16*)c.chunk_mat;
  __nv_bfloat16* opers = mats + units * 3 * RT_C * RT_C;
  float* factors = (float*)(opers + units * RC_NOPS * RT_C * D);
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(rec_channel_mats_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, rc_mats_smem(D));
    if (e == cudaSuccess) e = cudaFuncSetAttribute(rec_channel_chunk_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, rc_smem(D));
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  CUtensorMap tmX, tmM, tmK;
  int rc = cached_tmap_2d(&tmX, c.qkv, (uint64_t)T, (uint64_t)c.qkv_ld, 2, RT_C);
  if (rc == 0) rc = cached_tmap_2d(&tmM, mats, (uint64_t)units * 3 * RT_C, RT_C, 2, RT_C);
  if (rc == 0) rc = cached_tmap_2d(&tmK, opers, (uint64_t)units * RC_NOPS * RT_C, D, 2, RT_C);
  if (rc != 0) return rc;
  const dim3 g1((c.max_q_len + RT_C - 1) / RT_C, p.H, S), g2((p.V + 127) / 128, p.H, S);
  cudaError_t e = launch_pdl(rec_channel_mats_kernel<D>, g1, dim3(256), (size_t)rc_mats_smem(D), s, p, c, mats, opers, factors);
  if (e != cudaSuccess) return (int)e;
  return (int)launch_pdl(rec_channel_chunk_kernel<D>, g2, dim3(RC_THREADS), (size_t)rc_smem(D), s, tmX, tmM, tmK, p, c, (const float*)factors);
}

}  // namespace skein

// Bytes of chunk_mat for T rows of S sequences.
extern "C" long long skein_rec_channel_scratch_bytes(const SkeinRecParams* p, int T, int S) {
  using namespace skein;
  return rc_units(*p, T, S) * (3 * RT_MAT_BYTES + RC_NOPS * RT_C * p->D * 2 + rc_factors(p->D) * 4);
}

// After skein_rec_prep, in place of skein_rec_scan: bf16, D 64 or 128, V a multiple of 64; other sizes return -1.
extern "C" int skein_rec_channel(const SkeinRecParams* p, const SkeinRecChunk* c, int T, int S, void* stream) {
  using namespace skein;
  if (T == 0 || S == 0) return 0;
  if (p->kind != REC_CHANNEL || !p->step || !p->dt_bias || p->V % 64 != 0 || p->V < 64 || p->H % p->G != 0 || p->H > 65535 || S > 65535) return -1;
  if (c->qkv_ld % 8 != 0 || c->v_off % 8 != 0 || c->chunk_mat == nullptr || (uintptr_t)c->qkv % 16 != 0) return -1;
  cudaStream_t s = (cudaStream_t)stream;
  if (p->D == 64) return rec_channel_go<64>(*p, *c, T, S, s);
  return p->D == 128 ? rec_channel_go<128>(*p, *c, T, S, s) : -1;
}
