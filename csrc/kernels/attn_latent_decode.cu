// Attention of single rows over the latent cache on the 5th-generation tensor cores. All heads of a row share one cached row of
// kv_rank + rot elements per token, so the cached tokens (and then the latent's columns) fill the 128-row side of the MMA and
// the heads of the row, 16 or 32 per CTA, are its narrow side; more heads of a row read the cache through L2.
//
//   score[h, j] = (q_abs[h] . c_j + rot(q_rot[h]) . k_rot_j) * scale          out[h] = sum_j softmax(score)[h, j] c_j
//
// grid = (splits, head groups, rows); the splits of a row form a cluster. A CTA walks its tokens in tiles of 64, kept in shared
// memory as 64-column blocks of [64 tokens][128 bytes]:
//
//   warp 0      TMA producer: pages of the tile, two tiles in flight
//   warp 1      MMA issuer: S^T = C Q^T (tokens x heads, as the blocks land, spread over four accumulators that the softmax adds
//               up), and after the softmax O^T += C^T P^T, 128 latent columns at a time (the tile is the transposed A operand, P
//               comes from shared memory); the O products of a tile are issued between those of the next tile's scores
//   warps 2-5   softmax, thread = token: column maxima by halving exchanges inside a warp and a step through shared memory, P to
//               shared memory, per-thread partial sums; O is rescaled in tensor memory only when a maximum moved by more than 2^8
//
// At the end the CTA parks its unnormalised O in shared memory; every CTA of the cluster produces a share of the head rows, which
// one bulk copy per CTA pair brings to it. Every wait is bounded.
//
// q_abs holds the queries with the key expansion already applied; the rotated query part is rotated here, on its way to shared
// memory.
#include "attn_rule.cuh"
#include "ptx.cuh"
#include "launch.cuh"
#include <cuda.h>
#include <cuda_bf16.h>
#include <math.h>

namespace skein {

int cached_tmap_2d(CUtensorMap* out, const void* base, uint64_t rows, uint64_t k_elems, int elem_bytes, uint32_t box_rows);

constexpr int LD_THREADS = 192;
constexpr int LD_BN = 64;                            // tokens per tile
constexpr int LD_STAGES = 2;
constexpr int LD_CHUNK = LD_BN * 128;                // a 64-column block of a tile
constexpr int LD_MAX_GROUPS = 2;                     // groups of blocks with a barrier of their own: 256 latent columns each
constexpr int LD_MAX_SPLITS = 8;
constexpr int LD_ACC = 4;                            // accumulators of a score tile: a narrow product waits for the one it adds to, so
                                                     // neighbouring 16-element steps go to different ones and the softmax adds them up
constexpr int LD_TMEM_COLS = 512;
constexpr uint64_t LD_BUDGET_NS = 2000000000ull;

struct LatentDecodeParams {
  const __nv_bfloat16* q_abs;   // [T, H * K]
  const __nv_bfloat16* q;       // [T, q_ld], head h's rotated part at column h * (D + rot) + D
  const float* cos_sin;
  const int* positions;
  const int* seq_of_token;
  const int* block_table;
  __nv_bfloat16* out;           // [T, H * K]
  int* status;
  const float* sinks;           // [H] one more term exp(sinks[h]) in head h's denominator, or null
  long long q_ld;
  float scale_log2e;
  int H, D, rot, K, max_pos, max_blocks, num_pages, page_size, splits, nch, box_rows;
};

// byte offset of 16-byte chunk c of row r in 64-column blocks of [rows][128 bytes], 128-byte swizzle
__device__ __forceinline__ uint32_t ld_off(int r, int c, int rows) {
  return (uint32_t)((c >> 3) * rows * 128 + r * 128 + (((c & 7) ^ (r & 7)) << 4));
}
__device__ __forceinline__ void ld_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ void ld_cluster_sync() {
  asm volatile("barrier.cluster.arrive.release;\n\tbarrier.cluster.wait.acquire;" ::: "memory");
}
__device__ __forceinline__ uint32_t ld_map(uint32_t addr, uint32_t rank) {   // shared address of another CTA of the cluster
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
  return r;
}
// v[NH] per lane -> lane l returns the maximum (or sum) over the warp's lanes of element l mod NH, by halving exchanges
template <int NH, bool MAX>
__device__ __forceinline__ float ld_column_reduce(const float* v) {
  const int lane = threadIdx.x & 31;
  float a[NH];
#pragma unroll
  for (int i = 0; i < NH; ++i) a[i] = v[i];
  if (NH == 16) {
#pragma unroll
    for (int i = 0; i < NH; ++i) {
      const float o = __shfl_xor_sync(0xffffffffu, a[i], 16);
      a[i] = MAX ? fmaxf(a[i], o) : a[i] + o;
    }
  }
#pragma unroll
  for (int s = NH / 2; s > 0; s >>= 1) {
    const bool up = (lane & s) != 0;       // lanes with this bit keep the upper half
#pragma unroll
    for (int i = 0; i < s; ++i) {
      const float send = up ? a[i] : a[i + s], keep = up ? a[i + s] : a[i];
      const float o = __shfl_xor_sync(0xffffffffu, send, s);
      a[i] = MAX ? fmaxf(keep, o) : keep + o;
    }
  }
  return a[0];
}

template <int NH> __device__ __forceinline__ void ld_tmem_load(uint32_t addr, uint32_t* r) { if (NH == 32) tmem_ld32(addr, r); else tmem_ld16(addr, r); }

// NH: heads per CTA
template <int NH>
__global__ void __launch_bounds__(LD_THREADS, 1) attn_latent_decode_kernel(const __grid_constant__ CUtensorMap tmC, const LatentDecodeParams p) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t bar_full[LD_STAGES * LD_MAX_GROUPS], bar_empty[LD_STAGES * LD_MAX_GROUPS], bar_s[2], bar_p, bar_o, bar_r;
  __shared__ __align__(16) float m_s[NH];
  __shared__ float wred[4][NH], l_s[NH], alpha_s[NH];
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_flag;
  __shared__ int moved;
  pdl_trigger();
  pdl_wait();
  const int split = blockIdx.x, h0 = blockIdx.y * NH, t = blockIdx.z, ns = p.splits;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int K = p.K, nch = p.nch, park_ld = K + 4;
  const int ns_log = 31 - __clz(ns), rows_max = NH >> ns_log;       // splits: a power of two
  if (tid == 0) {
    abort_flag = 0;
    moved = 0;
    for (int c = 0; c < LD_STAGES * LD_MAX_GROUPS; ++c) { mbar_init(smem_u32(&bar_full[c]), 1); mbar_init(smem_u32(&bar_empty[c]), 1); }
    mbar_init(smem_u32(&bar_s[0]), 1); mbar_init(smem_u32(&bar_s[1]), 1); mbar_init(smem_u32(&bar_p), 128); mbar_init(smem_u32(&bar_o), 1); mbar_init(smem_u32(&bar_r), 1);
    fence_mbar_init();
  }
  if (tid >= 64 && tid - 64 < NH) { m_s[tid - 64] = -INFINITY; l_s[tid - 64] = 0.f; }
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
  const uint32_t q_s = base + LD_STAGES * nch * LD_CHUNK, p_s = q_s + nch * NH * 128;
  uint8_t* q_ptr = base_ptr + (q_s - base);
  uint8_t* p_ptr = base_ptr + (p_s - base);
  // queries -> shared memory (rows past H are zero), by everyone but the producer and ahead of the cache's tiles, behind which
  // they would queue: the latent part by asynchronous copies, the rotated part and the padding through registers (below)
  if (warp > 0) {
    for (int r = warp - 1; r < NH; r += LD_THREADS / 32 - 1) {
      const int h = h0 + r;
      const __nv_bfloat16* src = p.q_abs + (size_t)t * p.H * K + (size_t)(h < p.H ? h : 0) * K;
      for (int c = lane; c < K / 8; c += 32)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(q_s + ld_off(r, c, NH)), "l"(src + c * 8), "r"(h < p.H ? 16 : 0) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  if (p.seq_of_token == nullptr && tid == 0)     // the block table's first line, wanted as soon as the position is known
    asm volatile("prefetch.global.L2 [%0];" ::"l"(p.block_table + (size_t)t * p.max_blocks));
  int pos = p.positions[t];
  if (pos >= p.max_pos) { if (tid == 0) report_status(p.status, ST_BAD_INDEX, pos); pos = -1; }
  if (pos < 0) {      // padding row: the same decision in every CTA of the cluster
    if (split == 0)
      for (int i = tid; i < NH * K; i += LD_THREADS)
        if (h0 + i / K < p.H) p.out[(size_t)t * p.H * K + (size_t)h0 * K + i] = __float2bfloat16(0.f);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    return;
  }
  const int len = pos + 1, seq = p.seq_of_token ? p.seq_of_token[t] : t;
  const int per = ((len + 63) / 64 + ns - 1) / ns * 64;       // tokens of a split: whole 64-token pieces
  const int t0 = min(len, split * per), t1 = min(len, t0 + per);
  const int n_my = (t1 - t0 + LD_BN - 1) / LD_BN;
  const int nlat = (K + 63) / 64;                             // blocks that hold latent columns; the others only the rotated part
  const int nblk = (K + 127) / 128, ngrp = (nlat + 3) / 4;    // group g: blocks 4 g .. 4 g + 3, group 0 also the rotated-only blocks

  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_slot), LD_TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot, tm_o = tmem_slot + 2 * LD_ACC * 32;      // two buffers of S accumulators, then O

  if (warp > 0) {
    const int qt = tid - 32, kc = K / 8, rest = nch * 8 - kc;
    for (int i = qt; i < NH * rest; i += LD_THREADS - 32) {
      const int r = i / rest, c = kc + i % rest, col = c * 8 - K, h = h0 + r;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (h < p.H && col < p.rot) {
        const __nv_bfloat16* qr = p.q + (size_t)t * p.q_ld + (size_t)h * (p.D + p.rot) + p.D + col;
        const float2* cs = reinterpret_cast<const float2*>(p.cos_sin) + (size_t)pos * (p.rot / 2) + col / 2;
        __nv_bfloat162* vb = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float u = __bfloat162float(qr[2 * k]), w = __bfloat162float(qr[2 * k + 1]);
          const float2 a = cs[k];
          vb[k] = __floats2bfloat162_rn(u * a.x - w * a.y, w * a.x + u * a.y);
        }
      }
      *reinterpret_cast<uint4*>(q_ptr + ld_off(r, c, NH)) = v;
    }
  }

  if (warp == 0) {
    // ---------------------------------------------------------------- producer (one elected lane: the issue path stays uniform)
    if (elect_one()) {
      tma_prefetch_desc(&tmC);
      const uint64_t pol = l2_policy_evict_first();
      const int* bt = p.block_table + (size_t)seq * p.max_blocks;
      const int ps = p.page_size;
      bool ok = true;
      int armed = 0;      // blocks armed so far, in order
      for (int j = 0; j < n_my && ok; ++j) {
        const int tok0 = t0 + j * LD_BN, rows = min(t1 - tok0, LD_BN);
        const int boxes = (rows + p.box_rows - 1) / p.box_rows;
        int row_of[4];    // first cache row of every box of the tile
#pragma unroll
        for (int b = 0; b < 4; ++b) {
          if (b >= boxes) break;
          const int tok = tok0 + b * p.box_rows;
          int page = bt[tok / ps];
          if (page < 0 || page >= p.num_pages) { report_status(p.status, ST_BAD_INDEX, page); page = 0; }
          row_of[b] = page * ps + tok % ps;
        }
        const int s0 = j % LD_STAGES;
        for (int g = 0; g < ngrp; ++g) {
          const int c_hi = min(4 * g + 4, nlat), extra = g == 0 ? nch - nlat : 0, n = c_hi - 4 * g + extra;
          const uint32_t full = smem_u32(&bar_full[s0 * LD_MAX_GROUPS + g]);
          if (j >= LD_STAGES && !mbar_wait(smem_u32(&bar_empty[s0 * LD_MAX_GROUPS + g]), (j / LD_STAGES - 1) & 1, &abort_flag, LD_BUDGET_NS)) { ok = false; break; }
          mbar_expect_tx(full, (uint32_t)n * boxes * p.box_rows * 128);
          ++armed;
          for (int i = 0; i < n; ++i) {
            const int c = i < extra ? nlat + i : 4 * g + i - extra;
            for (int b = 0; b < boxes && b < 4; ++b)
              tma_load_2d(base + (s0 * nch + c) * LD_CHUNK + b * p.box_rows * 128, &tmC, full, c * 64, row_of[b], pol);
          }
        }
      }
      if (!ok) {
        abort_flag = 1;
        report_status(p.status, ST_TIMEOUT_SMEM_EMPTY, 30);
        volatile int never = 0;      // copies in flight still write this CTA's shared memory: wait for them (bounded)
        for (int a = max(0, armed - LD_STAGES * ngrp); a < armed; ++a) {
          const int j = a / ngrp;
          mbar_wait(smem_u32(&bar_full[(j % LD_STAGES) * LD_MAX_GROUPS + a % ngrp]), (j / LD_STAGES) & 1, &never, LD_BUDGET_NS);
        }
      }
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issuer (the queries are in shared memory: barrier 2)
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    fence_proxy_async_smem();
    asm volatile("bar.sync 2, 160;" ::: "memory");
    if (elect_one()) {
      const uint32_t idesc_s = umma_idesc(1, 1, LD_BN, NH);
      const uint32_t idesc_o = umma_idesc(1, 1, 128, NH) | (1u << 15);      // A operand MN-major: latent columns are contiguous
      bool ok = true;
      const uint64_t dp = umma_desc_sw128(p_s), da0 = umma_desc_sw128(base), dq0 = umma_desc_sw128(q_s);
      int done_o = 0;                   // tiles whose O products are issued
      auto issue_o = [&](int j) {
        tc_fence_after();
        const int s0 = j % LD_STAGES, k_steps = (min(t1 - (t0 + j * LD_BN), LD_BN) + 15) / 16;      // 16-token steps with a live token
        const uint64_t da = umma_desc_sw128_mn(base + s0 * nch * LD_CHUNK, LD_CHUNK);
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (k < k_steps)
#pragma unroll
            for (int b = 0; b < 4; ++b)      // neighbouring products add to different accumulators
              if (b < nblk) mma_f16(tm_o + b * NH, da + b * (2 * LD_CHUNK / 16) + k * (16 * 128 / 16), dp + 2 * k, idesc_o, (j > 0 || k > 0) ? 1u : 0u);
        for (int g = 0; g < ngrp; ++g) tc_commit(smem_u32(&bar_empty[s0 * LD_MAX_GROUPS + g]));
        tc_commit(smem_u32(&bar_o));
        done_o = j + 1;
      };
      for (int j = 0; j < n_my && ok; ++j) {
        const int s0 = j % LD_STAGES;
        const uint32_t d = tmem + (j & 1) * LD_ACC * 32;
        for (int g = 0; g < ngrp; ++g) {
          // while waiting for the group: the previous tile's O as soon as its P is there, which frees that tile's memory
          const uint32_t full = smem_u32(&bar_full[s0 * LD_MAX_GROUPS + g]);
          if (done_o < j) {
            const uint64_t w0 = global_timer_ns();
            bool landed = false;
            while (!landed && done_o < j) {
              landed = mbar_test_wait(full, (j / LD_STAGES) & 1);
              if (mbar_test_wait(smem_u32(&bar_p), (j - 1) & 1)) issue_o(j - 1);
              else if (!landed && (abort_flag != 0 || global_timer_ns() - w0 > LD_BUDGET_NS)) break;      // the wait below reports it
            }
          }
          if (!mbar_wait(full, (j / LD_STAGES) & 1, &abort_flag, LD_BUDGET_NS)) { ok = false; break; }
          tc_fence_after();
          // descriptors count in 16-byte units: a 16-element step is 2
          const uint64_t da = da0 + (uint32_t)(s0 * nch) * (LD_CHUNK / 16);
          if (g == 0)
            for (int c = nlat; c < nch; ++c)
#pragma unroll
              for (int k = 0; k < 4; ++k)
                mma_f16(d + k * 32, da + c * (LD_CHUNK / 16) + 2 * k, dq0 + c * (NH * 128 / 16) + 2 * k, idesc_s, c > nlat ? 1u : 0u);
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int c = 4 * g + i;
            if (c >= nlat) break;
            if (i == 2 && done_o < j && mbar_test_wait(smem_u32(&bar_p), (j - 1) & 1)) issue_o(j - 1);
#pragma unroll
            for (int k = 0; k < 4; ++k)
              mma_f16(d + k * 32, da + c * (LD_CHUNK / 16) + 2 * k, dq0 + c * (NH * 128 / 16) + 2 * k, idesc_s, (c > 0 || nch > nlat) ? 1u : 0u);
          }
        }
        if (!ok) break;
        tc_commit(smem_u32(&bar_s[j & 1]));
        if (done_o < j) {
          if (!mbar_wait(smem_u32(&bar_p), (j - 1) & 1, &abort_flag, LD_BUDGET_NS)) { ok = false; break; }
          issue_o(j - 1);
        }
      }
      if (ok && n_my > 0) {
        if (mbar_wait(smem_u32(&bar_p), (n_my - 1) & 1, &abort_flag, LD_BUDGET_NS)) issue_o(n_my - 1);
        else ok = false;
      }
      if (!ok && abort_flag == 0) { abort_flag = 1; report_status(p.status, ST_TIMEOUT_SMEM_FULL, 31); }
    }
  } else {
    const int st = tid - 64, lane_grp = warp & 3;
    const uint32_t lane_addr = (uint32_t)(lane_grp * 32) << 16;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    fence_proxy_async_smem();
    asm volatile("bar.sync 2, 160;" ::: "memory");
    const int r = lane_grp * 32 + lane;             // tensor-memory lane = latent column of a block of O
    const int tok = lane_grp * 16 + lane;           // a 64-row product keeps 16 rows in the first lanes of every warp's 32
    float lp[NH];                                   // this thread's share of the heads' sums
#pragma unroll
    for (int i = 0; i < NH; ++i) lp[i] = 0.f;
    bool ok = true;
    for (int j = 0; j < n_my; ++j) {
      if (!mbar_wait(smem_u32(&bar_s[j & 1]), (j >> 1) & 1, &abort_flag, LD_BUDGET_NS)) ok = false;     // carries on: no barrier below is skipped
      tc_fence_after();
      const bool live = lane < 16 && t0 + j * LD_BN + tok < t1;
      float x[NH];
      {
        uint32_t sv[2][NH];
        const uint32_t sa = tmem + (j & 1) * LD_ACC * 32 + lane_addr;
#pragma unroll
        for (int i = 0; i < NH; ++i) x[i] = 0.f;
#pragma unroll
        for (int a = 0; a < LD_ACC; a += 2) {
          ld_tmem_load<NH>(sa + a * 32, sv[0]);
          ld_tmem_load<NH>(sa + a * 32 + 32, sv[1]);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < NH; ++i) x[i] += __uint_as_float(sv[0][i]) + __uint_as_float(sv[1][i]);
        }
#pragma unroll
        for (int i = 0; i < NH; ++i) x[i] = live ? x[i] * p.scale_log2e : -INFINITY;
      }
      const float wm = ld_column_reduce<NH, true>(x);
      if (lane < NH) wred[lane_grp][lane] = wm;
      ld_sync();
      if (st < NH) {
        const float mx = fmaxf(fmaxf(wred[0][st], wred[1][st]), fmaxf(wred[2][st], wred[3][st])), m = m_s[st];
        // a tile holds at least one live token; the maximum only moves by more than 2^8 (the sums stay exact in the end)
        const float mn = (m == -INFINITY || mx > m + 8.f) ? fmaxf(m, mx) : m;
        alpha_s[st] = m == -INFINITY ? 1.f : exp2f(m - mn);
        if (m != -INFINITY && mn != m) moved = j + 1;
        m_s[st] = mn;
      }
      ld_sync();
      if (j > 0 && !mbar_wait(smem_u32(&bar_o), (j - 1) & 1, &abort_flag, LD_BUDGET_NS)) ok = false;
      if (moved == j + 1) {
        tc_fence_after();
        for (int b = 0; b < nblk; ++b) {
          uint32_t ov[NH];
          ld_tmem_load<NH>(tm_o + lane_addr + b * NH, ov);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < NH; ++i) ov[i] = __float_as_uint(__uint_as_float(ov[i]) * alpha_s[i]);
#pragma unroll
          for (int c = 0; c < NH; c += 16) tmem_st16(tm_o + lane_addr + b * NH + c, ov + c);
        }
        tmem_st_wait();
#pragma unroll
        for (int i = 0; i < NH; ++i) lp[i] *= alpha_s[i];
      }
      if (lane < 16) {
        uint8_t* pr = p_ptr + (tok & 7) * 2;         // P[h][token], token-contiguous rows of 128 bytes
        const int pc = tok >> 3;
#pragma unroll
        for (int i = 0; i < NH; i += 4) {            // the maxima first: loads do not wait behind the stores below
          const float4 m4 = *reinterpret_cast<const float4*>(m_s + i);
          x[i] = exp2f(x[i] - m4.x); x[i + 1] = exp2f(x[i + 1] - m4.y); x[i + 2] = exp2f(x[i + 2] - m4.z); x[i + 3] = exp2f(x[i + 3] - m4.w);
        }
#pragma unroll
        for (int i = 0; i < NH; ++i) {
          const __nv_bfloat16 pb = __float2bfloat16(x[i]);
          lp[i] += __bfloat162float(pb);
          *reinterpret_cast<__nv_bfloat16*>(pr + i * 128 + ((pc ^ (i & 7)) << 4)) = pb;
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(smem_u32(&bar_p));
    }
    // ---- sums, then O from tensor memory to its parking place (fp32, over the tiles' memory): [producer][rows][park_ld] ----
    const float ws = ld_column_reduce<NH, false>(lp);
    if (lane < NH) wred[lane_grp][lane] = ws;
    ld_sync();
    if (st < NH) l_s[st] = wred[0][st] + wred[1][st] + wred[2][st] + wred[3][st];
    if (n_my > 0 && !mbar_wait(smem_u32(&bar_o), (n_my - 1) & 1, &abort_flag, LD_BUDGET_NS)) ok = false;
    if (!ok && abort_flag == 0) { abort_flag = 1; report_status(p.status, ST_TIMEOUT_TMEM_FULL, 32); }
    tc_fence_after();
    float* park = reinterpret_cast<float*>(base_ptr);
    for (int b = 0; b < nblk; ++b) {
      uint32_t ov[NH];
      if (n_my > 0) { ld_tmem_load<NH>(tm_o + lane_addr + b * NH, ov); tmem_ld_wait(); }
      const int d = b * 128 + r;
      if (d < K)
#pragma unroll
        for (int i = 0; i < NH; ++i) park[((i & (ns - 1)) * rows_max + (i >> ns_log)) * park_ld + d] = n_my > 0 ? __uint_as_float(ov[i]) : 0.f;
    }
    if (st < NH) {       // a row's maximum and sum ride in its last four floats
      float* pm = park + ((st & (ns - 1)) * rows_max + (st >> ns_log)) * park_ld + K;
      pm[0] = m_s[st]; pm[1] = l_s[st];
    }
    fence_proxy_async_smem();
  }
  tc_fence_before();
  // ---- exchange: CTA c of the cluster produces the head rows i with i mod splits = c. Behind the barrier the tiles' memory is dead
  // in every CTA, and one bulk copy per producer brings a CTA's share of its rows there ----
  const uint32_t block_bytes = (uint32_t)(rows_max * park_ld * 4);
  const uint32_t recv = base + (uint32_t)(ns * rows_max * park_ld * 4);                  // [split][rows][park_ld]
  if (ns > 1) ld_cluster_sync(); else __syncthreads();
  if (tid == 0 && ns > 1) {
    mbar_expect_tx(smem_u32(&bar_r), (uint32_t)(ns - 1) * block_bytes);
    for (int c = 0; c < ns; ++c)
      if (c != split)
        asm volatile("cp.async.bulk.shared::cluster.shared::cta.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                     ::"r"(ld_map(recv + split * block_bytes, c)), "r"(base + c * block_bytes), "r"(block_bytes), "r"(ld_map(smem_u32(&bar_r), c)) : "memory");
  }
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, LD_TMEM_COLS);
  }
  if (ns > 1 && !mbar_wait(smem_u32(&bar_r), 0, &abort_flag, LD_BUDGET_NS) && tid == 0) report_status(p.status, ST_TIMEOUT_SPLITK, split);
  // this CTA's rows are here: it reads no other CTA's memory from now on (the wait for the others is at the end)
  if (ns > 1) asm volatile("barrier.cluster.arrive.release;" ::: "memory");
  __syncthreads();
  for (int row = warp; row < rows_max; row += LD_THREADS / 32) {
    const int h = h0 + row * ns + split;
    if (h >= p.H) break;
    // lane c: split c's maximum and sum of this row, then the weight of its O: exp2(m_c - M) / sum_c exp2(m_c - M) l_c
    auto part = [&](int c) -> const float* {
      return reinterpret_cast<const float*>(base_ptr + ((c == split ? base + c * block_bytes : recv + c * block_bytes) - base)) + row * park_ld;
    };
    float mc = -INFINITY, lc = 0.f;
    if (lane < ns) { const float* q = part(lane) + K; mc = q[0]; lc = q[1]; }
    float M = mc;
#pragma unroll
    for (int o = LD_MAX_SPLITS / 2; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
    float w = mc == -INFINITY ? 0.f : exp2f(mc - M), L = w * lc;
#pragma unroll
    for (int o = LD_MAX_SPLITS / 2; o > 0; o >>= 1) L += __shfl_xor_sync(0xffffffffu, L, o);
    w *= attn_norm(M, L, attn_sink_log2(p.sinks, h));
    __nv_bfloat16* orow = p.out + (size_t)t * p.H * K + (size_t)h * K;
    for (int c0 = 0; c0 < K; c0 += 512) {            // four groups of 4 columns per lane in flight
      float4 acc[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) acc[u] = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int c = 0; c < ns; ++c) {
        const float wc = __shfl_sync(0xffffffffu, w, c);
        const float* q = part(c) + c0 + lane * 4;
#pragma unroll
        for (int u = 0; u < 4; ++u)
          if (c0 + lane * 4 + u * 128 < K) {
            const float4 v = *reinterpret_cast<const float4*>(q + u * 128);
            acc[u].x += wc * v.x; acc[u].y += wc * v.y; acc[u].z += wc * v.z; acc[u].w += wc * v.w;
          }
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int col = c0 + lane * 4 + u * 128;
        if (col >= K) continue;
        const __nv_bfloat162 a = __floats2bfloat162_rn(acc[u].x, acc[u].y), b = __floats2bfloat162_rn(acc[u].z, acc[u].w);
        uint2 o2;
        o2.x = *reinterpret_cast<const uint32_t*>(&a); o2.y = *reinterpret_cast<const uint32_t*>(&b);
        *reinterpret_cast<uint2*>(orow + col) = o2;
      }
    }
  }
  if (ns > 1) asm volatile("barrier.cluster.wait.acquire;" ::: "memory");      // nobody leaves while its memory is being read
}

template <int NH>
static int latent_decode_launch(const CUtensorMap& tm, LatentDecodeParams& p, int T, int groups, cudaStream_t s) {
  size_t smem = (size_t)p.nch * (LD_STAGES * LD_CHUNK + NH * 128) + NH * 128 + 1024 + 64;
  // the operands of the last block reach past the tiles: that memory (unused results) must exist
  const size_t reach = (size_t)(LD_STAGES * p.nch + 2) * LD_CHUNK + 1024, park = (size_t)2 * NH * (p.K + 4) * 4 + 1024;
  if (reach > smem) smem = reach;
  if (park > smem) smem = park;
  if (smem > 222 * 1024) return -1;
  auto fn = attn_latent_decode_kernel<NH>;
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 222 * 1024);
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  cudaLaunchConfig_t cfg;
  memset(&cfg, 0, sizeof(cfg));
  cfg.gridDim = dim3(p.splits, groups, T);
  cfg.blockDim = dim3(LD_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = p.splits; attr[1].val.clusterDim.y = 1; attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  return (int)cudaLaunchKernelEx(&cfg, fn, tm, p);
}

}  // namespace skein

// Returns 0, a cudaError_t, or -1 for shapes this kernel does not take (the caller then uses the plain kernel): kv_rank and rot
// multiples of 8, kv_rank <= 512, page size 16, 32 or a multiple of 64. splits 0: chosen from the row count and ctx_hint.
extern "C" int skein_latent_attn_decode(const void* q_abs, const void* q, long long q_ld, const float* cos_sin, int max_pos,
                                        const int* positions, const int* seq_of_token, const int* block_table, int max_blocks,
                                        const void* cache, int num_pages, int page_size, void* out, int T, int H, int D, int rot, int kv_rank,
                                        float scale, const float* sinks, int splits, int ctx_hint, int* status, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (kv_rank % 8 || rot % 8 || kv_rank < 8 || kv_rank > 512 || rot < 8 || T > 65535 || scale <= 0.f) return -1;
  if (!(page_size == 16 || page_size == 32 || page_size % 64 == 0)) return -1;
  LatentDecodeParams p;
  p.q_abs = (const __nv_bfloat16*)q_abs; p.q = (const __nv_bfloat16*)q; p.cos_sin = cos_sin; p.positions = positions;
  p.seq_of_token = seq_of_token; p.block_table = block_table; p.out = (__nv_bfloat16*)out; p.status = status; p.q_ld = q_ld;
  p.sinks = sinks;
  p.scale_log2e = scale * 1.4426950408889634f;
  p.H = H; p.D = D; p.rot = rot; p.K = kv_rank; p.max_pos = max_pos; p.max_blocks = max_blocks; p.num_pages = num_pages; p.page_size = page_size;
  p.nch = (kv_rank + rot + 63) / 64;
  const int nh = H <= 16 ? 16 : 32, groups = (H + nh - 1) / nh;
  p.box_rows = page_size < 64 ? page_size : 64;
  int dev = 0, sms = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms <= 0) sms = 148;
  if (splits <= 0) {
    splits = sms / (T * groups > 0 ? T * groups : 1);
    if (splits > ctx_hint / LD_BN) splits = ctx_hint / LD_BN;
  }
  p.splits = 1;                       // a power of two, so that the head rows divide evenly among the cluster's CTAs
  while (p.splits * 2 <= splits && p.splits < LD_MAX_SPLITS) p.splits *= 2;
  CUtensorMap tm;
  const int rc = cached_tmap_2d(&tm, cache, (uint64_t)num_pages * page_size, (uint64_t)(kv_rank + rot), 2, p.box_rows);
  if (rc != 0) return rc;
  return nh == 16 ? latent_decode_launch<16>(tm, p, T, groups, (cudaStream_t)stream) : latent_decode_launch<32>(tm, p, T, groups, (cudaStream_t)stream);
}
