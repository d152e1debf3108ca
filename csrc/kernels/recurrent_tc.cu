// The recurrences of recurrent.cu over whole chunks of 64 tokens on the tensor cores (bf16 models, D = 64 or 128, V a multiple
// of 64). With G_i the running sum of the log decays inside a chunk, S the state before it and r_q, r_k the factors that make
// unit vectors (1 where there are none):
//
//   U   = T diag(beta) (V - diag(e^G r_k) K S)          delta; T = (I + A)^-1, A_ij = beta_i k_i.k_j r_k r_k e^(G_i - G_j), j < i
//   U   = V                                             otherwise
//   O   = diag(e^G r_q) Q S + P U,                      P_ij = q_i.k_j r_q r_k e^(G_i - G_j) [coef_j], j <= i
//   S  <- e^G_last S + (diag(e^(G_last - G) r_k [coef]) K)^T U
//
//   rec_tc_mats   every chunk and head at once: T (as a sum of two bf16 matrices), P, the factors per token
//   rec_tc_chunk  one CTA per (128 columns of V, head, sequence) walks the chunks. Everything is computed transposed, so that
//                 a column of V is a tensor-memory lane and a thread: the left operands (S, U and what is derived from them)
//                 go from registers to tensor memory, the right ones are the K, Q, T and P tiles that TMA brought to shared
//                 memory, as they lie there.
//                     warp 0      TMA, two chunks in flight         warp 1   MMA issue (one lane)
//                     warps 2-9   two threads per lane: half of the state's rows (fp32 registers) and half of the tokens each
//
// The state is fp32 from chunk to chunk. As an operand it is split into two bf16 summands (hi + lo, 16 bits of mantissa), and so
// is everything that flows back into it; q, k and v are exact. The read-out's second product takes P and U in bf16, as attention
// takes its weights. Every wait is bounded. Compiled without fast-math.
#include "ptx.cuh"
#include "launch.cuh"
#include "recurrent.cuh"
#include "recurrent_tc.cuh"
#include <cuda.h>
#include <cuda_bf16.h>
#include <math.h>

namespace skein {

int cached_tmap_2d(CUtensorMap* out, const void* base, uint64_t rows, uint64_t k_elems, int elem_bytes, uint32_t box_rows);

constexpr int RT_SC = 5 * RT_C;                // floats of a chunk's factors: beta | e^G r_k | e^G r_q | e^(G_last - G) r_k coef | e^G_last

// ---- the chunks' matrices ---------------------------------------------------------------------------
__host__ __device__ constexpr int rt_kq_bytes(int d) { return 2 * RT_C * (d + 8) * 2; }
// K and Q, whose place X and Y take later; then A
__host__ __device__ constexpr int rt_mats_smem(int d, bool delta) {
  return (!delta || rt_kq_bytes(d) > 2 * RT_C * RT_LX * 2 + 2 * 32 * RT_LY * 2 ? rt_kq_bytes(d) : 2 * RT_C * RT_LX * 2 + 2 * 32 * RT_LY * 2) +
         (delta ? 2 * RT_C * RT_LX * 2 + RT_C * RT_LD * 4 : 0);
}

constexpr int RT_HB = 8;         // most heads of a CTA

// grid (chunks, H / heads, S), 256 threads: `heads` heads that share queries and keys, whose products are computed once
template <int D, bool DELTA>
__global__ void __launch_bounds__(256, 3) rec_tc_mats_kernel(const RecParams p, const RecChunk c, __nv_bfloat16* mats, float* factors, int heads) {
  extern __shared__ __align__(16) uint8_t mt_smem[];
  __shared__ __align__(16) float Gh_all[RT_HB][RT_C];
  __shared__ __align__(16) float Gl_all[RT_HB][RT_C];
  __shared__ __align__(16) float coef_all[RT_HB][RT_C];
  __shared__ __align__(16) float rq_s[RT_C], rk_s[RT_C];
  pdl_trigger();
  pdl_wait();
  const int h0 = blockIdx.y * heads, seq = blockIdx.z, len = c.q_len[seq], i0 = blockIdx.x * RT_C;
  if (i0 >= len) return;
  const int n = min(RT_C, len - i0), q_start = c.q_start[seq], t0 = q_start + i0;
  const int unit0 = (rt_chunk0(q_start, seq) + blockIdx.x) * p.H + h0;
  const int grp = h0 / (p.H / p.G), gd = p.G * D, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  constexpr int LD = D + 8;
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(mt_smem);
  __nv_bfloat16* q_s = k_s + RT_C * LD;
  __nv_bfloat16* Xh = k_s;                                   // [64][RT_LX], once K and Q are done with
  __nv_bfloat16* Xl = Xh + RT_C * RT_LX;
  __nv_bfloat16* Yh = Xl + RT_C * RT_LX;                     // [32][RT_LY]
  __nv_bfloat16* Yl = Yh + 32 * RT_LY;
  __nv_bfloat16* Ah = reinterpret_cast<__nv_bfloat16*>(mt_smem + rt_mats_smem(D, true) - 2 * RT_C * RT_LX * 2 - RT_C * RT_LD * 4);
  __nv_bfloat16* Al = Ah + RT_C * RT_LX;
  float* Ad = reinterpret_cast<float*>(Al + RT_C * RT_LX);   // [64][RT_LD] the 16 x 16 blocks on the diagonal
  for (int i = tid; i < RT_C * (D / 8) * 2; i += 256) {
    const int m = i / (RT_C * (D / 8)), r = i % (RT_C * (D / 8)) / (D / 8), ch = i % (D / 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < n) v = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)c.qkv + (size_t)(t0 + r) * c.qkv_ld + (m ? 0 : gd) + grp * D + ch * 8);
    *reinterpret_cast<uint4*>((m ? q_s : k_s) + r * LD + ch * 8) = v;
  }
  if (tid < RT_C) {
    const float* un = DELTA ? c.unit + (size_t)(t0 + (tid < n ? tid : 0)) * 2 * p.G : nullptr;
    rq_s[tid] = DELTA ? un[grp] : 1.f;
    rk_s[tid] = DELTA ? un[p.G + grp] : 1.f;
  }
  if (warp < heads) {      // a warp per head: running sum of the log decays, whose differences must keep the accuracy of 32-bit
    const float2* gt = reinterpret_cast<const float2*>(c.gates) + h0 + warp;
    const float2 g0 = 2 * lane < n ? gt[(size_t)(t0 + 2 * lane) * p.H] : make_float2(0.f, 0.f);
    const float2 g1 = 2 * lane + 1 < n ? gt[(size_t)(t0 + 2 * lane + 1) * p.H] : make_float2(0.f, 0.f);
    double a = g0.x, b = g1.x, s = a + b;
    for (int o = 1; o < 32; o <<= 1) { const double u = __shfl_up_sync(0xffffffffu, s, o); if (lane >= o) s += u; }
    const double before = __shfl_up_sync(0xffffffffu, s, 1);
    a += lane > 0 ? before : 0.0;
    b += a;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const double g = (e ? b : a) * 1.4426950408889634;      // base 2 from here
      Gh_all[warp][2 * lane + e] = (float)g;
      Gl_all[warp][2 * lane + e] = (float)(g - (double)(float)g);
      coef_all[warp][2 * lane + e] = e ? g1.y : g0.y;
    }
  }
  __syncthreads();
  // K K^T by warps 0-3 and Q K^T by warps 4-7 (without K K^T: two warps per 16 rows of Q K^T), 16 rows each
  const bool qk = !DELTA || warp >= 4;
  const int blk = warp & 3, r0 = 16 * blk, nb0 = DELTA ? 0 : 4 * (warp >> 2);
  constexpr int nbn = DELTA ? 8 : 4;
  float prod[nbn][4];
#pragma unroll
  for (int i = 0; i < nbn; ++i) prod[i][0] = prod[i][1] = prod[i][2] = prod[i][3] = 0.f;
  {
    const uint32_t a_base = smem_u32(qk ? q_s : k_s), b_base = smem_u32(k_s);
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) {
      uint32_t a[4];
      rt_ldsm4(a_base + ((r0 + (lane & 15)) * LD + ks * 16 + (lane >> 4) * 8) * 2, a);
#pragma unroll
      for (int nb = 0; nb < nbn; nb += 2) {
        if ((nb0 + nb) * 8 > r0 + 15) continue;       // above the diagonal
        const int mat = lane >> 3;
        uint32_t b[4];
        rt_ldsm4(b_base + (((nb0 + nb) * 8 + (mat >> 1) * 8 + (lane & 7)) * LD + ks * 16 + (mat & 1) * 8) * 2, b);
        rt_mma(prod[nb], a, b[0], b[1]);
        rt_mma(prod[nb + 1], a, b[2], b[3]);
      }
    }
  }
  for (int hh = 0; hh < heads; ++hh) {
    const float *Gh_s = Gh_all[hh], *Gl_s = Gl_all[hh], *coef_s = coef_all[hh];
    auto decay = [&](int i, int j) { return exp2f((Gh_s[i] - Gh_s[j]) + (Gl_s[i] - Gl_s[j])); };      // e^(G_i - G_j)
    const int unit = unit0 + hh;
    float* f = factors + (size_t)unit * RT_SC;
    if (tid < RT_C) {
      const float eg = exp2f(Gh_s[tid]);
      f[tid] = DELTA ? coef_s[tid] : 1.f;
      f[RT_C + tid] = eg * rk_s[tid];
      f[2 * RT_C + tid] = eg * rq_s[tid];
      f[3 * RT_C + tid] = tid < n ? decay(n - 1, tid) * rk_s[tid] * (DELTA ? 1.f : coef_s[tid]) : 0.f;
      f[4 * RT_C + tid] = exp2f(Gh_s[n - 1]);
    }
    __nv_bfloat16* out = mats + (size_t)unit * (DELTA ? 3 : 1) * RT_C * RT_C;
    if (DELTA && hh > 0) __syncthreads();        // the previous head's X has been read
    float gi[2], gl[2], ri[2];                   // of this thread's two rows
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int i = r0 + (lane >> 2) + 8 * hf;
      gi[hf] = Gh_s[i];
      gl[hf] = Gl_s[i];
      ri[hf] = i < n ? (qk ? rq_s[i] : rk_s[i] * coef_s[i]) : 0.f;
    }
#pragma unroll
    for (int nb = 0; nb < nbn; ++nb) {
      const int j = (nb0 + nb) * 8 + (lane & 3) * 2;
      const bool below = (nb0 + nb) * 8 <= r0 + 15;
      float2 gj = make_float2(0.f, 0.f), glj = gj, rj = gj;
      if (below) {
        gj = *reinterpret_cast<const float2*>(Gh_s + j);
        glj = *reinterpret_cast<const float2*>(Gl_s + j);
        rj = *reinterpret_cast<const float2*>(rk_s + j);
        if (!DELTA) { const float2 cj = *reinterpret_cast<const float2*>(coef_s + j); rj.x *= cj.x; rj.y *= cj.y; }
      }
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int i = r0 + (lane >> 2) + 8 * hf;
        float v[2] = {0.f, 0.f};
        if (below) {
          const int last = qk ? i : i - 1;       // last column of the row
          if (j <= last) v[0] = prod[nb][2 * hf] * exp2f((gi[hf] - gj.x) + (gl[hf] - glj.x)) * rj.x * ri[hf];
          if (j + 1 <= last) v[1] = prod[nb][2 * hf + 1] * exp2f((gi[hf] - gj.y) + (gl[hf] - glj.y)) * rj.y * ri[hf];
        }
        if (qk) {
          *reinterpret_cast<uint32_t*>(out + (DELTA ? 2 : 0) * RT_C * RT_C + i * RT_C + j) = rt_pack(v[0], v[1]);
        } else if (nb >> 1 == blk) {
          Ad[i * RT_LD + (j & 15)] = v[0];
          Ad[i * RT_LD + (j & 15) + 1] = v[1];
        } else if (nb >> 1 < blk) {
          uint32_t hi, lo;
          rt_split(v[0], v[1], hi, lo);
          *reinterpret_cast<uint32_t*>(Ah + i * RT_LX + j) = hi;
          *reinterpret_cast<uint32_t*>(Al + i * RT_LX + j) = lo;
        }
      }
    }
    if (!DELTA) continue;
    __syncthreads();
    rt_invert(Ad, Ah, Xh, Xl, Yh, Yl);
    for (int i = tid; i < 2 * RT_C * 8; i += 256) {
      const int m = i / (RT_C * 8), r = i % (RT_C * 8) / 8, ch = i % 8;
      reinterpret_cast<uint4*>(out)[i] = *reinterpret_cast<const uint4*>((m ? Xl : Xh) + r * RT_LX + ch * 8);
    }
  }
}

// ---- the walk over the chunks -------------------------------------------------------------------------
constexpr int RT_THREADS = 320, RT_COMPUTE = 256;
__host__ __device__ constexpr int rt_stage_bytes(int d, bool delta, bool pair) {   // [K | Q] per 64 columns, V, matrices, factors
  return d / 64 * 2 * RT_C * 128 + 2 * RT_C * 128 + (delta ? 3 : pair ? 2 : 1) * RT_MAT_BYTES + 3072;
}
constexpr int RT_OUT_BYTES = RT_C * 256;      // a chunk's outputs, [64][128] bf16
__host__ __device__ constexpr int rt_smem(int d, bool delta, bool pair) { return 2 * (rt_stage_bytes(d, delta, pair) + RT_OUT_BYTES) + 1024 + 256; }

// PAIR (no correction, V = 64): the tile's two halves are two neighbouring heads of a group, each with its own P and factors.
//
// tensor-memory columns. delta: A operands S (hi, lo), U'; accumulators [R | O1] of one product, U, O2, dS.
constexpr uint32_t TM_SH = 0, TM_SL = 64, TM_R = 128, TM_O1 = 192, TM_U = 256, TM_O2 = 320, TM_DS = 384;

template <int D, bool DELTA, bool PAIR>
__global__ void __launch_bounds__(RT_THREADS, 1)
rec_tc_chunk_kernel(const __grid_constant__ CUtensorMap tmX, const __grid_constant__ CUtensorMap tmM, const RecParams p, const RecChunk c,
                    const float* factors) {
  constexpr int HALVES = D / 64, KQ_HALF = 2 * RT_C * 128, STAGE = rt_stage_bytes(D, DELTA, PAIR), NMAT = DELTA ? 3 : PAIR ? 2 : 1;
  constexpr int MATS = DELTA ? 3 : 1;            // of one head
  constexpr int OFF_V = HALVES * KQ_HALF, OFF_M = OFF_V + 2 * RT_C * 128, OFF_F = OFF_M + NMAT * RT_MAT_BYTES;
  const int h = blockIdx.y * (PAIR ? 2 : 1), seq = blockIdx.z, tile0 = blockIdx.x * 128;
  const int len = c.q_len[seq], slot = p.slots[seq];
  if (len < 1 || slot < 0 || slot >= p.num_slots) return;
  const int t0 = c.q_start[seq], n_chunks = (len + RT_C - 1) / RT_C, unit0 = rt_chunk0(t0, seq);
  const int grp = h / (p.H / p.G), gd = p.G * D;

  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
  const uint32_t bars = base + 2 * (STAGE + RT_OUT_BYTES);
  const uint32_t bar_full = bars, bar_empty = bars + 16, bar_s = bars + 32, bar_r = bars + 40, bar_rr = bars + 48, bar_u = bars + 56,
                 bar_ur = bars + 64, bar_o = bars + 72;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(base_ptr + 2 * (STAGE + RT_OUT_BYTES) + 96);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(base_ptr + 2 * (STAGE + RT_OUT_BYTES) + 104);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    for (int s = 0; s < 2; ++s) { mbar_init(bar_full + 8 * s, 1); mbar_init(bar_empty + 8 * s, RT_COMPUTE); }
    mbar_init(bar_s, RT_COMPUTE); mbar_init(bar_r, 1); mbar_init(bar_rr, RT_COMPUTE); mbar_init(bar_u, 1); mbar_init(bar_ur, RT_COMPUTE);
    mbar_init(bar_o, 1);
    abort_flag[0] = 0;
    abort_flag[1] = 0;      // never set: the drain waits of a failing producer run out on their time budget only
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tm = *tmem_slot;
  const int width = PAIR ? 128 : p.V;             // columns of V from tile0's head on
  const int v_halves = min(2, (width - tile0 + 63) / 64);

  if (warp == 0) {
    // ---------------------------------------------------------------- TMA producer
    if (lane == 0) {
      tma_prefetch_desc(&tmX);
      tma_prefetch_desc(&tmM);
      const uint64_t pol = l2_policy_evict_first(), pol_keep = l2_policy_evict_last();
      const uint32_t bytes = HALVES * KQ_HALF + v_halves * RT_C * 128 + NMAT * RT_MAT_BYTES + (PAIR ? 2 : 1) * RT_SC * 4;
      bool ok = true;
      int armed[2] = {0, 0};
      for (int j = 0; j < n_chunks; ++j) {
        const int s = j & 1;
        if (j >= 2 && !mbar_wait(bar_empty + 8 * s, ((j >> 1) - 1) & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
        const uint32_t st = base + s * STAGE, full = bar_full + 8 * s;
        mbar_expect_tx(full, bytes);
        ++armed[s];
        const int row = t0 + j * RT_C, unit = (unit0 + j) * p.H + h;
        for (int hf = 0; hf < HALVES; ++hf) {
          tma_load_2d(st + hf * KQ_HALF, &tmX, full, gd + grp * D + hf * 64, row, pol_keep);
          tma_load_2d(st + hf * KQ_HALF + RT_C * 128, &tmX, full, grp * D + hf * 64, row, pol_keep);
        }
        for (int hf = 0; hf < v_halves; ++hf) tma_load_2d(st + OFF_V + hf * RT_C * 128, &tmX, full, c.v_off + h * p.V + tile0 + hf * 64, row, pol);
        for (int m = 0; m < NMAT; ++m) tma_load_2d(st + OFF_M + m * RT_MAT_BYTES, &tmM, full, 0, (unit * MATS + m) * RT_C, pol);
        bulk_load_1d(st + OFF_F, factors + (size_t)unit * RT_SC, (PAIR ? 2 : 1) * RT_SC * 4, full);
      }
      if (!ok) {
        if (*abort_flag == 0) { *abort_flag = 1; report_status(p.status, ST_TIMEOUT_SMEM_EMPTY, 20); }
        // copies already issued still write this CTA's shared memory: wait for them (bounded) before leaving
        for (int s = 0; s < 2; ++s)
          if (armed[s] > 0) mbar_wait(bar_full + 8 * s, (armed[s] - 1) & 1, abort_flag + 1, RT_BUDGET_NS);
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
        ok = mbar_wait(bar_full + 8 * s, (j >> 1) & 1, abort_flag, RT_BUDGET_NS) && mbar_wait(bar_s, j & 1, abort_flag, RT_BUDGET_NS);
        if (!ok) break;
        tc_fence_after();
        // [R | O1] = S [K | Q]^T (without R: Q only)
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int k = 0; k < D / 16; ++k) {
            const uint32_t b = st + (k >> 2) * KQ_HALF + (k & 3) * 32 + (DELTA ? 0 : RT_C * 128);
            mma_f16_ts(tm + (DELTA ? TM_R : TM_O1), tm + (part ? TM_SL : TM_SH) + k * 8, umma_desc_sw128(b), DELTA ? id_2c : id_c,
                       part > 0 || k > 0 ? 1u : 0u);
          }
        if (PAIR) tc_commit(bar_r);
        if (DELTA) {
          tc_commit(bar_r);
          ok = mbar_wait(bar_rr, j & 1, abort_flag, RT_BUDGET_NS);
          if (!ok) break;
          tc_fence_after();
          // U = R T^T; R (hi, lo) lies where O2 will go
#pragma unroll
          for (int part = 0; part < 3; ++part)
#pragma unroll
            for (int k = 0; k < RT_C / 16; ++k)
              mma_f16_ts(tm + TM_U, tm + TM_O2 + (part == 1 ? 32 : 0) + k * 8, umma_desc_sw128(st + OFF_M + (part == 2 ? RT_MAT_BYTES : 0) + k * 32), id_c,
                         part > 0 || k > 0 ? 1u : 0u);
          tc_commit(bar_u);
          ok = mbar_wait(bar_ur, j & 1, abort_flag, RT_BUDGET_NS);
          if (!ok) break;
          tc_fence_after();
        }
        // O2 = U P^T, dS = U' K. Operands: U in R's columns and U' in S's (delta), U in its own and U' in R's (otherwise)
#pragma unroll
        for (int k = 0; k < RT_C / 16; ++k)
          mma_f16_ts(tm + TM_O2, tm + (DELTA ? TM_R : TM_U) + k * 8, umma_desc_sw128(st + OFF_M + (MATS - 1) * RT_MAT_BYTES + k * 32), id_c, k > 0 ? 1u : 0u);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int k = 0; k < RT_C / 16; ++k)
            mma_f16_ts(tm + TM_DS, tm + (DELTA ? TM_SH : TM_R) + part * 32 + k * 8, umma_desc_sw128_mn(st + k * 16 * 128, KQ_HALF), id_d,
                       part > 0 || k > 0 ? 1u : 0u);
        if (PAIR) {
          // the second head's O2 takes the place of S as an operand, whose product has to be complete
          ok = mbar_wait(bar_r, j & 1, abort_flag, RT_BUDGET_NS);
          if (!ok) break;
          tc_fence_after();
#pragma unroll
          for (int k = 0; k < RT_C / 16; ++k) mma_f16_ts(tm + TM_SH, tm + TM_U + k * 8, umma_desc_sw128(st + OFF_M + RT_MAT_BYTES + k * 32), id_c, k > 0 ? 1u : 0u);
        }
        tc_commit(bar_o);
      }
      if (!ok && *abort_flag == 0) { *abort_flag = 1; report_status(p.status, ST_TIMEOUT_SMEM_FULL, 21); }
    }
  } else {
    // ---------------------------------------------------------------- state, splits, outputs: thread <-> column of V, half hf
    const int quarter = warp & 3, hf = (warp - 2) >> 2, v = quarter * 32 + lane, col = PAIR ? v & 63 : tile0 + v;
    const int second = PAIR ? v >> 6 : 0, head = h + second;
    const uint32_t ta = tm + ((uint32_t)(quarter * 32) << 16);
    const bool in = col < p.V;
    constexpr int NS = D / 2;               // rows of the state in this thread
    float* S = p.state + ((size_t)slot * p.H + head) * D * p.V + (size_t)hf * NS * p.V + col;
    const bool fresh = p.positions[t0] == 0;
    float s[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) s[i] = (in && !fresh) ? S[(size_t)i * p.V] : 0.f;
    const float skip = p.skip ? p.skip[head] : 0.f;
    auto put_state = [&]() {                // S as an operand, hi and lo
#pragma unroll
      for (int b = 0; b < NS / 32; ++b) {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) rt_split(s[b * 32 + 2 * i], s[b * 32 + 2 * i + 1], hi[i], lo[i]);
        tmem_st16(ta + TM_SH + hf * (NS / 2) + b * 16, hi);
        tmem_st16(ta + TM_SL + hf * (NS / 2) + b * 16, lo);
      }
    };
    const uint32_t v_byte = (uint32_t)(v & 63) * 2;
    const uint32_t v_half = OFF_V + (v >> 6) * RT_C * 128;
    const int cols = min(128, width - tile0), ct = tid - 64;      // columns of the tile; number of this thread among the 256
    // V[token i][col] of a stage; 128-byte rows, 16-byte pieces swizzled by the row
    auto value = [&](int sg, int i) {
      return __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(base_ptr + sg * STAGE + v_half + i * 128 + (v_byte ^ ((i & 7) << 4))));
    };
    auto factor = [&](int sg) { return reinterpret_cast<const float*>(base_ptr + sg * STAGE + OFF_F) + second * RT_SC; };
    // what chunk j's first products read: S, and without a correction U = V (exact) and U' = V times its factor
    auto open_chunk = [&](int j) {
      put_state();
      if (!DELTA) {
        const int sg = j & 1;
        if (!mbar_wait(bar_full + 8 * sg, (j >> 1) & 1, abort_flag, RT_BUDGET_NS)) return false;
        const float* f = factor(sg);
        uint32_t u[16], hi[16], lo[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int t = hf * 32 + 2 * i;
          const float a = value(sg, t), b = value(sg, t + 1);
          u[i] = rt_pack(a, b);
          rt_split(a * f[3 * RT_C + t], b * f[3 * RT_C + t + 1], hi[i], lo[i]);
        }
        tmem_st16(ta + TM_U + hf * 16, u);
        tmem_st16(ta + TM_R + hf * 16, hi);
        tmem_st16(ta + TM_R + 32 + hf * 16, lo);
      }
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(bar_s);
      return true;
    };
    bool ok = open_chunk(0);
    for (int j = 0; j < n_chunks && ok; ++j) {
      const int sg = j & 1, n = min(RT_C, len - j * RT_C);
      const float* f = factor(sg);
      if (DELTA) {
        if (!mbar_wait(bar_full + 8 * sg, (j >> 1) & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
        uint32_t r[32], hi[16], lo[16];
        float x[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) x[i] = value(sg, hf * 32 + i);       // (while the product runs)
        if (!mbar_wait(bar_r, j & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
        tc_fence_after();
        tmem_ld32(ta + TM_R + hf * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int t = hf * 32 + 2 * i;
          const float2 b2 = *reinterpret_cast<const float2*>(f + t), e2 = *reinterpret_cast<const float2*>(f + RT_C + t);
          rt_split(b2.x * (x[2 * i] - e2.x * __uint_as_float(r[2 * i])), b2.y * (x[2 * i + 1] - e2.y * __uint_as_float(r[2 * i + 1])), hi[i], lo[i]);
        }
        tmem_st16(ta + TM_O2 + hf * 16, hi);
        tmem_st16(ta + TM_O2 + 32 + hf * 16, lo);
        tmem_st_wait();
        tc_fence_before();
        mbar_arrive(bar_rr);
        if (!mbar_wait(bar_u, j & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
        tc_fence_after();
        uint32_t u[16];
        tmem_ld32(ta + TM_U + hf * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int t = hf * 32 + 2 * i;
          const float2 s2 = *reinterpret_cast<const float2*>(f + 3 * RT_C + t);
          const float a = __uint_as_float(r[2 * i]), b = __uint_as_float(r[2 * i + 1]);
          u[i] = rt_pack(a, b);
          rt_split(a * s2.x, b * s2.y, hi[i], lo[i]);
        }
        tmem_st16(ta + TM_R + hf * 16, u);
        tmem_st16(ta + TM_SH + hf * 16, hi);
        tmem_st16(ta + TM_SH + 32 + hf * 16, lo);
        tmem_st_wait();
        tc_fence_before();
        mbar_arrive(bar_ur);
      }
      if (!mbar_wait(bar_o, j & 1, abort_flag, RT_BUDGET_NS)) { ok = false; break; }
      tc_fence_after();
      uint32_t o[16];                       // the chunk's outputs of this thread, pairs of tokens
      {
        uint32_t o1[32], o2[32];
        tmem_ld32(ta + TM_O1 + hf * 32, o1);
        tmem_ld32(ta + (second ? TM_SH : TM_O2) + hf * 32, o2);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int t = hf * 32 + 2 * i;
          const float2 e2 = *reinterpret_cast<const float2*>(f + 2 * RT_C + t);
          float a = fmaf(e2.x, __uint_as_float(o1[2 * i]), __uint_as_float(o2[2 * i]));
          float b = fmaf(e2.y, __uint_as_float(o1[2 * i + 1]), __uint_as_float(o2[2 * i + 1]));
          if (!DELTA) { a = fmaf(skip, value(sg, t), a); b = fmaf(skip, value(sg, t + 1), b); }
          o[i] = rt_pack(a, b);
        }
      }
      const float keep = f[4 * RT_C];
#pragma unroll
      for (int b = 0; b < NS / 32; ++b) {
        uint32_t d[32];
        tmem_ld32(ta + TM_DS + hf * NS + b * 32, d);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) s[b * 32 + i] = fmaf(keep, s[b * 32 + i], __uint_as_float(d[i]));
      }
      tc_fence_before();
      mbar_arrive(bar_empty + 8 * sg);
      if (j + 1 < n_chunks) ok = open_chunk(j + 1);
      // the outputs go through shared memory to whole 16-byte pieces of the rows, while the next chunk's product runs. Two buffers:
      // a thread can be one chunk ahead of another here, not two.
      uint8_t* ob = base_ptr + 2 * STAGE + (j & 1) * RT_OUT_BYTES;
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
      report_status(p.status, ST_TIMEOUT_TMEM_FULL, 22);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tm, 512);
  }
}

template <int D, bool DELTA, bool PAIR>
static int rec_tc_go(const RecParams& p, const RecChunk& c, int T, int S, cudaStream_t s) {
  const int units = (T / RT_C + S + 1) * p.H, nmat = DELTA ? 3 : 1;
  __nv_bfloat16* mats = (__nv_bfloat16*)c.chunk_mat;
  float* factors = (float*)(mats + (size_t)units * nmat * RT_C * RT_C);
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(rec_tc_mats_kernel<D, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, rt_mats_smem(D, DELTA));
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(rec_tc_chunk_kernel<D, DELTA, PAIR>, cudaFuncAttributeMaxDynamicSharedMemorySize, rt_smem(D, DELTA, PAIR));
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  CUtensorMap tmX, tmM;
  int rc = cached_tmap_2d(&tmX, c.qkv, (uint64_t)T, (uint64_t)c.qkv_ld, 2, RT_C);
  if (rc == 0) rc = cached_tmap_2d(&tmM, mats, (uint64_t)units * nmat * RT_C, RT_C, 2, RT_C);
  if (rc != 0) return rc;
  int heads = RT_HB;                            // of a CTA of the first kernel: a power of two that divides the heads of a group
  while ((p.H / p.G) % heads != 0) heads /= 2;
  const dim3 g1((c.max_q_len + RT_C - 1) / RT_C, p.H / heads, S), g2(PAIR ? 1 : (p.V + 127) / 128, PAIR ? p.H / 2 : p.H, S);
  cudaError_t e = launch_pdl(rec_tc_mats_kernel<D, DELTA>, g1, dim3(256), (size_t)rt_mats_smem(D, DELTA), s, p, c, mats, factors, heads);
  if (e != cudaSuccess) return (int)e;
  return (int)launch_pdl(rec_tc_chunk_kernel<D, DELTA, PAIR>, g2, dim3(RT_THREADS), (size_t)rt_smem(D, DELTA, PAIR), s, tmX, tmM, p, c,
                         (const float*)factors);
}

}  // namespace skein

// Bytes of chunk_mat for T rows of S sequences.
extern "C" long long skein_rec_tc_scratch_bytes(const SkeinRecParams* p, int T, int S) {
  using namespace skein;
  return (long long)(T / RT_C + S + 1) * p->H * ((p->kind == REC_DELTA ? 3 : 1) * RT_MAT_BYTES + RT_SC * 4);
}

// After skein_rec_prep, in place of skein_rec_scan: bf16, D 64 or 128, V a multiple of 64; other sizes return -1.
extern "C" int skein_rec_tc(const SkeinRecParams* p, const SkeinRecChunk* c, int T, int S, void* stream) {
  using namespace skein;
  if (T == 0 || S == 0) return 0;
  if ((p->D != 64 && p->D != 128) || p->V % 64 != 0 || p->V < 64 || p->H % p->G != 0 || p->H > 65535 || S > 65535) return -1;
  if (c->qkv_ld % 8 != 0 || c->v_off % 8 != 0 || c->chunk_mat == nullptr || (uintptr_t)c->qkv % 16 != 0) return -1;
  cudaStream_t s = (cudaStream_t)stream;
  if (p->kind == REC_DELTA) return p->D == 64 ? rec_tc_go<64, true, false>(*p, *c, T, S, s) : rec_tc_go<128, true, false>(*p, *c, T, S, s);
  if (p->V == 64 && (p->H / p->G) % 2 == 0)
    return p->D == 64 ? rec_tc_go<64, false, true>(*p, *c, T, S, s) : rec_tc_go<128, false, true>(*p, *c, T, S, s);
  return p->D == 64 ? rec_tc_go<64, false, false>(*p, *c, T, S, s) : rec_tc_go<128, false, false>(*p, *c, T, S, s);
}
