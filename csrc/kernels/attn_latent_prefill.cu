// Causal attention of latent-attention prefill chunks on the 5th-generation tensor cores, with keys and values expanded per
// head beforehand (one GEMM over the chunk's context). A score is the sum of two products: the unrotated parts (per-head
// keys) and the rotated parts (one key part shared by all heads, read from the context rows themselves).
//
// One CTA = 256 query rows of one head as two tiles of 128, walking the context in 128-token tiles:
//
//   warp 0      TMA producer: both Q tiles once, then per context tile the keys (unrotated chunks from the expanded matrix,
//               the rotated chunk from the context rows) and the values; single K and V buffers, refilled while the other
//               operand is in use. Head sizes need not be whole 64-element chunks: a box past the head reads zeros.
//   warp 1      MMA issuer: S_t = Q_t K^T and O_t += P_t V for the two tiles in turn (S and O in tensor memory, P taken from
//               tensor memory), ordered so that one tile's softmax runs while the other tile's products do:
//                   P0 V, S0 of the next context tile, P1 V, S1 of the next context tile
//   warps 2-5   softmax of tile 0 (thread = query row), warps 6-9 of tile 1; the last step normalises, multiplies by the
//               sigmoid of the output gate if there is one, and stores
//
// S0 | S1 | O0 | O1 take all 512 tensor-memory columns, Q, K and V up to 176 KB of shared memory: one CTA per SM. Every wait is
// bounded; on expiry the CTA records a status code, waits for its copies in flight, frees its tensor memory and returns.
#include "attn_rule.cuh"
#include "ptx.cuh"
#include "launch.cuh"
#include <cuda.h>
#include <cuda_bf16.h>
#include <math.h>

namespace skein {

int cached_tmap_2d(CUtensorMap* out, const void* base, uint64_t rows, uint64_t k_elems, int elem_bytes, uint32_t box_rows);
int cached_tmap_heads(CUtensorMap* out, const void* base, uint64_t rows, uint64_t heads, uint64_t d, uint64_t head_stride,
                      uint64_t row_stride, uint32_t box_rows);

constexpr int LP_BM = 128, LP_BN = 128;
constexpr int LP_THREADS = 320;
constexpr int LP_CHUNK = 128 * 128;                  // 128 rows x 64 elements
constexpr uint64_t LP_BUDGET_NS = 4000000000ull;

struct LatentPrefillParams {
  const int* q_start;       // [S] first row of the sequence's chunk in q / out
  const int* q_len;         // [S]
  const int* kv_len;        // [S] tokens of context including the chunk
  const int* ctx_start;     // [S] first context row of the sequence
  const __nv_bfloat16* gate;
  __nv_bfloat16* out;       // [T, H * V]
  const float* sinks;       // [H] one more term exp(sinks[h]) in head h's denominator, or null
  int* status;
  int gate_ld;
  int H, D, rot, V, kv_rank;
  int dc, vc;               // 64-element chunks of the unrotated part and of the values
  float scale_log2e;
};

__global__ void __launch_bounds__(LP_THREADS, 1)
attn_latent_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                           const __grid_constant__ CUtensorMap tmR, const __grid_constant__ CUtensorMap tmV, const LatentPrefillParams p) {
  pdl_trigger();
  pdl_wait();
  const int qt = (int)gridDim.x - 1 - (int)blockIdx.x;     // long rows first: the causal work grows with the row
  const int head = blockIdx.y, seq = blockIdx.z;
  const int qlen = p.q_len[seq];
  const int q0 = qt * 2 * LP_BM;
  if (q0 >= qlen) return;
  const int kvlen = p.kv_len[seq];
  const int pos0 = kvlen - qlen;
  const int qrow0 = p.q_start[seq], crow0 = p.ctx_start[seq];
  const bool two = q0 + LP_BM < qlen;
  const int hi0 = min(kvlen, pos0 + min(q0 + LP_BM, qlen));                    // exclusive bound of the keys tile 0 / 1 sees
  const int hi1 = two ? min(kvlen, pos0 + min(q0 + 2 * LP_BM, qlen)) : 0;
  const int n0 = (hi0 + LP_BN - 1) / LP_BN, n1 = (hi1 + LP_BN - 1) / LP_BN;
  const int N = max(n0, n1);

  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
  const uint32_t qk_bytes = (p.dc + 1) * LP_CHUNK, v_bytes = p.vc * LP_CHUNK;
  const uint32_t q_s = base, k_s = base + 2 * qk_bytes, v_s = k_s + qk_bytes, bars = v_s + v_bytes;
  const uint32_t bar_q = bars, bar_kfull = bars + 8, bar_kempty = bars + 16, bar_vfull = bars + 24, bar_vempty = bars + 32;
  const uint32_t bar_s = bars + 40, bar_p = bars + 56, bar_o = bars + 72;      // one per tile, 8 bytes apart
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(base_ptr + (bars - base) + 96);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(base_ptr + (bars - base) + 104);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    mbar_init(bar_q, 1); mbar_init(bar_kfull, 1); mbar_init(bar_kempty, 1); mbar_init(bar_vfull, 1); mbar_init(bar_vempty, 1);
    for (int t = 0; t < 2; ++t) { mbar_init(bar_s + 8 * t, 1); mbar_init(bar_p + 8 * t, 128); mbar_init(bar_o + 8 * t, 1); }
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
  const uint32_t tmem = *tmem_slot;

  if (warp == 0) {
    // ---------------------------------------------------------------- TMA producer
    if (elect_one()) {
      const uint64_t pol_q = l2_policy_evict_first(), pol_kv = l2_policy_evict_last();
      mbar_expect_tx(bar_q, (two ? 2 : 1) * qk_bytes);
      for (int t = 0; t < (two ? 2 : 1); ++t) {
        const int row = qrow0 + q0 + t * LP_BM;
        for (int c = 0; c < p.dc; ++c) tma_load_3d(q_s + t * qk_bytes + c * LP_CHUNK, &tmQ, bar_q, c * 64, head, row, pol_q);
        tma_load_3d(q_s + t * qk_bytes + p.dc * LP_CHUNK, &tmQ, bar_q, p.D, head, row, pol_q);
      }
      bool ok = true;
      int armed_k = 0, armed_v = 0;
      for (int j = 0; j < N && ok; ++j) {
        const int row = crow0 + j * LP_BN;
        if (j > 0 && !mbar_wait(bar_kempty, (j - 1) & 1, abort_flag, LP_BUDGET_NS)) { ok = false; break; }
        mbar_expect_tx(bar_kfull, qk_bytes);
        ++armed_k;
        for (int c = 0; c < p.dc; ++c) tma_load_3d(k_s + c * LP_CHUNK, &tmK, bar_kfull, c * 64, head, row, pol_kv);
        tma_load_2d(k_s + p.dc * LP_CHUNK, &tmR, bar_kfull, p.kv_rank, row, pol_kv);
        if (j > 0 && !mbar_wait(bar_vempty, (j - 1) & 1, abort_flag, LP_BUDGET_NS)) { ok = false; break; }
        mbar_expect_tx(bar_vfull, v_bytes);
        ++armed_v;
        for (int c = 0; c < p.vc; ++c) tma_load_3d(v_s + c * LP_CHUNK, &tmV, bar_vfull, c * 64, head, row, pol_kv);
      }
      if (!ok) {
        if (*abort_flag == 0) { *abort_flag = 1; report_status(p.status, ST_TIMEOUT_SMEM_EMPTY, 20); }
        // copies already issued still write this CTA's shared memory: wait for them (bounded) before leaving
        mbar_wait(bar_q, 0, abort_flag + 1, LP_BUDGET_NS);
        if (armed_k > 0) mbar_wait(bar_kfull, (armed_k - 1) & 1, abort_flag + 1, LP_BUDGET_NS);
        if (armed_v > 0) mbar_wait(bar_vfull, (armed_v - 1) & 1, abort_flag + 1, LP_BUDGET_NS);
      }
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issuer (one elected lane: the issue path stays uniform)
    if (elect_one()) {
      const uint32_t idesc_s = umma_idesc(1, 1, LP_BM, LP_BN);
      const uint32_t idesc_o = umma_idesc(1, 1, LP_BM, p.vc * 64) | (1u << 16);      // B operand MN-major
      const int dsteps = (p.D + 15) / 16, rsteps = (p.rot + 15) / 16;
      const uint64_t dq0 = umma_desc_sw128(q_s), dk0 = umma_desc_sw128(k_s), dv0 = umma_desc_sw128_mn(v_s, LP_CHUNK);
      auto issue_s = [&](int t) {
        const uint32_t d = tmem + t * 128;
        // descriptors count in 16-byte units: a 16-element step is 2, a 64-element block LP_CHUNK / 16
        const uint64_t dq = dq0 + (t ? qk_bytes / 16 : 0);
#pragma unroll
        for (int k = 0; k < 8; ++k)
          if (k < dsteps) mma_f16(d, dq + (k >> 2) * (LP_CHUNK / 16) + (k & 3) * 2, dk0 + (k >> 2) * (LP_CHUNK / 16) + (k & 3) * 2, idesc_s, k > 0 ? 1u : 0u);
        const uint32_t ro = p.dc * (LP_CHUNK / 16);
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (k < rsteps) mma_f16(d, dq + ro + k * 2, dk0 + ro + k * 2, idesc_s, 1u);
        tc_commit(bar_s + 8 * t);
      };
      auto issue_o = [&](int t, int j, int hi) {
        const int k_steps = (min(hi, (j + 1) * LP_BN) - j * LP_BN + 15) / 16;       // 16-token steps with a visible key
#pragma unroll
        for (int k = 0; k < 8; ++k)
          if (k < k_steps) mma_f16_ts(tmem + 256 + t * 128, tmem + t * 128 + k * 8, dv0 + k * (16 * 128 / 16), idesc_o, (j > 0 || k > 0) ? 1u : 0u);
        tc_commit(bar_o + 8 * t);
      };
      bool ok = mbar_wait(bar_q, 0, abort_flag, LP_BUDGET_NS) && mbar_wait(bar_kfull, 0, abort_flag, LP_BUDGET_NS);
      if (ok) {
        tc_fence_after();
        issue_s(0);
        if (n1 > 0) issue_s(1);
        tc_commit(bar_kempty);
      }
      for (int j = 0; j < N && ok; ++j) {
        if (!mbar_wait(bar_vfull, j & 1, abort_flag, LP_BUDGET_NS)) { ok = false; break; }
        if (j < n0) {
          if (!mbar_wait(bar_p, j & 1, abort_flag, LP_BUDGET_NS)) { ok = false; break; }
          tc_fence_after();
          issue_o(0, j, hi0);
        }
        if (j + 1 < N) {
          if (!mbar_wait(bar_kfull, (j + 1) & 1, abort_flag, LP_BUDGET_NS)) { ok = false; break; }
          tc_fence_after();
          if (j + 1 < n0) issue_s(0);
        }
        if (j < n1) {
          if (!mbar_wait(bar_p + 8, j & 1, abort_flag, LP_BUDGET_NS)) { ok = false; break; }
          tc_fence_after();
          issue_o(1, j, hi1);
        }
        tc_commit(bar_vempty);
        if (j + 1 < N) {
          if (j + 1 < n1) issue_s(1);
          tc_commit(bar_kempty);
        }
      }
      if (!ok && *abort_flag == 0) { *abort_flag = 1; report_status(p.status, ST_TIMEOUT_SMEM_FULL, 21); }
    }
  } else {
    // ---------------------------------------------------------------- softmax warps: thread <-> query row of tile t
    const int t = warp >= 6 ? 1 : 0;
    const int n_tiles = t ? n1 : n0, hi = t ? hi1 : hi0;
    const int lane_grp = warp & 3;                      // the 32 tensor-memory lanes this warp may access
    const int r = lane_grp * 32 + lane;                 // row of the tile
    const uint32_t lane_addr = (uint32_t)(lane_grp * 32) << 16;
    const uint32_t tm_s = tmem + t * 128 + lane_addr, tm_o = tmem + 256 + t * 128 + lane_addr;
    const int row0 = q0 + t * LP_BM;                    // chunk row of the tile's first query
    int pos_r = pos0 + row0 + r;
    if (pos_r > kvlen - 1) pos_r = kvlen - 1;           // rows past the chunk are computed, finite, and never stored
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      const int c0 = j * LP_BN;
      if (!mbar_wait(bar_s + 8 * t, j & 1, abort_flag, LP_BUDGET_NS)) { ok = false; break; }
      tc_fence_after();
      const bool masked = c0 + LP_BN - 1 > pos0 + row0;   // some row of the tile sees only part of these keys
      const int limit = pos_r - c0;                       // this row sees columns 0 .. limit of the tile
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int h = 0; h < LP_BN / 64; ++h) {
        uint32_t sv[64];
        tmem_ld32(tm_s + h * 64, sv);
        tmem_ld32(tm_s + h * 64 + 32, sv + 32);
        tmem_ld_wait();
        if (masked) {
#pragma unroll
          for (int i = 0; i < 64; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], (h * 64 + i <= limit) ? __uint_as_float(sv[i]) : -INFINITY);
        } else {
#pragma unroll
          for (int i = 0; i < 64; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sv[i]));
        }
      }
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * p.scale_log2e;    // the scale is positive
      // the running maximum only moves when the tile's maximum exceeds it by more than 2^8 (see attn_prefill_tc.cu)
      const float m_new = (m == -INFINITY || mx > m + 8.f) ? fmaxf(m, mx) : m;
      const float alpha = (m == -INFINITY) ? 1.f : exp2f(m - m_new);
      if (j > 0) {
        if (!mbar_wait(bar_o + 8 * t, (j - 1) & 1, abort_flag, LP_BUDGET_NS)) { ok = false; break; }
        tc_fence_after();
        if (__any_sync(0xffffffffu, alpha != 1.f)) {
          for (int h = 0; h < p.vc; ++h) {
            uint32_t ov[64];
            tmem_ld32(tm_o + h * 64, ov);
            tmem_ld32(tm_o + h * 64 + 32, ov + 32);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 64; ++i) ov[i] = __float_as_uint(__uint_as_float(ov[i]) * alpha);
#pragma unroll
            for (int c = 0; c < 4; ++c) tmem_st16(tm_o + h * 64 + c * 16, ov + c * 16);
          }
        }
      }
      l *= alpha;
      m = m_new;
      float rs = 0.f;
#pragma unroll
      for (int h = 0; h < LP_BN / 64; ++h) {
        uint32_t sv[64];
        tmem_ld32(tm_s + h * 64, sv);
        tmem_ld32(tm_s + h * 64 + 32, sv + 32);
        tmem_ld_wait();
        uint32_t pk[32];
#pragma unroll
        for (int i = 0; i < 64; i += 2) {
          float x0 = fmaf(__uint_as_float(sv[i]), p.scale_log2e, -m_new);
          float x1 = fmaf(__uint_as_float(sv[i + 1]), p.scale_log2e, -m_new);
          if (masked) {
            if (h * 64 + i > limit) x0 = -INFINITY;
            if (h * 64 + i + 1 > limit) x1 = -INFINITY;
          }
          // the row sum is taken over the rounded values, the ones the tensor cores multiply
          const __nv_bfloat162 pb = __floats2bfloat162_rn(exp2f(x0), exp2f(x1));
          const float2 pf = __bfloat1622float2(pb);
          rs += pf.x + pf.y;
          pk[i >> 1] = *reinterpret_cast<const uint32_t*>(&pb);
        }
        // columns [32 h, 32 h + 32) of P lie inside columns [0, 64 h + 64) of S, all of which have been read
        tmem_st16(tm_s + h * 32, pk);
        tmem_st16(tm_s + h * 32 + 16, pk + 16);
      }
      l += rs;
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(bar_p + 8 * t);
    }
    (void)hi;
    if (n_tiles > 0) {
      if (ok && mbar_wait(bar_o + 8 * t, (n_tiles - 1) & 1, abort_flag, LP_BUDGET_NS)) {
        tc_fence_after();
        const float inv = attn_norm(m, l, attn_sink_log2(p.sinks, head));
        const bool store = row0 + r < qlen;
        const size_t row = (size_t)(qrow0 + row0 + r);
        __nv_bfloat16* orow = p.out + row * ((size_t)p.H * p.V) + (size_t)head * p.V;
        const __nv_bfloat16* grow = p.gate ? p.gate + row * p.gate_ld + (size_t)head * p.V : nullptr;
        for (int c = 0; c < p.vc * 4; ++c) {
          uint32_t ov[16];
          tmem_ld16(tm_o + c * 16, ov);
          tmem_ld_wait();
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int col = c * 16 + half * 8;
            if (!store || col >= p.V) continue;
            float g[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) g[i] = inv;
            if (grow) {
              const uint4 gv = *reinterpret_cast<const uint4*>(grow + col);
              const __nv_bfloat162* gb = reinterpret_cast<const __nv_bfloat162*>(&gv);
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                const float2 f = __bfloat1622float2(gb[i]);
                g[2 * i] *= 1.f / (1.f + __expf(-f.x)); g[2 * i + 1] *= 1.f / (1.f + __expf(-f.y));
              }
            }
            uint32_t pk[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const __nv_bfloat162 b = __floats2bfloat162_rn(__uint_as_float(ov[half * 8 + 2 * i]) * g[2 * i],
                                                             __uint_as_float(ov[half * 8 + 2 * i + 1]) * g[2 * i + 1]);
              pk[i] = *reinterpret_cast<const uint32_t*>(&b);
            }
            *reinterpret_cast<uint4*>(orow + col) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
          }
        }
      } else if (*abort_flag == 0) {
        *abort_flag = 1;
        report_status(p.status, ST_TIMEOUT_TMEM_FULL, 22);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

}  // namespace skein

// q [q_rows, q_ld] (rotated), dense [ctx_rows, L] context rows with the rotated key part in the last `rot` columns, kv [ctx_rows,
// H * (D + V)] expanded keys then values, out [q_rows, H * V]. D, V <= 128, rot <= 64, all multiples of 8.
extern "C" int skein_latent_attn_prefill(const void* q, long long q_ld, int q_rows, const void* dense, int L, const void* kv, int ctx_rows,
                                         const void* gate, int gate_ld, const int* q_start, const int* q_len, const int* kv_len,
                                         const int* ctx_start, void* out, int* status, int S, int max_q_len, int H, int D, int rot, int V,
                                         float scale, const float* sinks, void* stream) {
  using namespace skein;
  if (S == 0 || max_q_len == 0) return 0;
  if (D < 1 || D > 128 || V < 1 || V > 128 || rot < 1 || rot > 64 || D % 8 || V % 8 || rot % 8 || q_ld % 8 || L % 8 || L <= rot || scale <= 0.f) return -1;
  if (gate != nullptr && (gate_ld % 8 || ((uintptr_t)gate & 15))) return -1;
  LatentPrefillParams p;
  p.q_start = q_start; p.q_len = q_len; p.kv_len = kv_len; p.ctx_start = ctx_start; p.gate = (const __nv_bfloat16*)gate;
  p.out = (__nv_bfloat16*)out; p.sinks = sinks; p.status = status; p.gate_ld = gate_ld; p.H = H; p.D = D; p.rot = rot; p.V = V; p.kv_rank = L - rot;
  p.dc = (D + 63) / 64; p.vc = (V + 63) / 64; p.scale_log2e = scale * 1.4426950408889634f;
  CUtensorMap tmQ, tmK, tmR, tmV;
  int rc = cached_tmap_heads(&tmQ, q, q_rows, H, D + rot, D + rot, q_ld, LP_BM);
  if (rc == 0) rc = cached_tmap_heads(&tmK, kv, ctx_rows, H, D, D, (uint64_t)H * (D + V), LP_BN);
  if (rc == 0) rc = cached_tmap_heads(&tmV, (const __nv_bfloat16*)kv + (size_t)H * D, ctx_rows, H, V, V, (uint64_t)H * (D + V), LP_BN);
  if (rc == 0) rc = cached_tmap_2d(&tmR, dense, ctx_rows, L, 2, LP_BN);
  if (rc != 0) return rc;
  const size_t smem = (size_t)(3 * (p.dc + 1) + p.vc) * LP_CHUNK + 1024 + 256;
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(attn_latent_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 11 * LP_CHUNK + 1280);
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  const dim3 grid((max_q_len + 2 * LP_BM - 1) / (2 * LP_BM), H, S);
  return (int)launch_pdl(attn_latent_prefill_kernel, grid, dim3(LP_THREADS), smem, (cudaStream_t)stream, tmQ, tmK, tmR, tmV, p);
}
