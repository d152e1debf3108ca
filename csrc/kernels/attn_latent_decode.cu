// Attention of single rows over the latent cache: all heads of a row share one cached row of kv_rank + rot elements per token,
// so the heads are the rows of the MMA tile and every cached byte is read once per 16 / 32 / 64 heads.
//
//   score[h, j] = (q_abs[h] . c_j + rot(q_rot[h]) . k_rot_j) * scale          out[h] = sum_j softmax(score)[h, j] c_j
//
// grid = (splits, head groups, rows); the splits of a row form a cluster. A CTA has 8 compute warps and a producer warp that
// streams tiles of 32 or 64 tokens (whole pages or parts of one, 128-byte swizzle, TMA) into a ring. Per tile:
//   S = Q C^T      a warp owns 8 tokens and one or two 16-head tiles, over all of kv_rank + rot
//   softmax        in shared memory, a warp owns whole head rows; P in bf16
//   O += P C       a warp owns an eighth of the kv_rank columns for all heads of the group, accumulators in registers
// The splits' results are merged through distributed shared memory: every CTA of the cluster parks its unnormalised O with its
// maxima and sums, and merges a share of the head rows from all of them. Every wait of the ring is bounded.
//
// q_abs holds the queries with the key expansion already applied; the rotated query part is rotated here, on its way to shared
// memory. Products run on mma.sync m16n8k16 (bf16, fp32 accumulation): with few heads the kernel is bound by the cache's bytes.
#include "ptx.cuh"
#include "launch.cuh"
#include <cuda.h>
#include <cuda_bf16.h>
#include <math.h>

namespace skein {

int cached_tmap_2d(CUtensorMap* out, const void* base, uint64_t rows, uint64_t k_elems, int elem_bytes, uint32_t box_rows);

constexpr int LD_WARPS = 8;
constexpr int LD_THREADS = (LD_WARPS + 1) * 32;
constexpr int LD_MAX_STAGES = 6;
constexpr int LD_MAX_SPLITS = 8;
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
  long long q_ld;
  float scale_log2e;
  int H, D, rot, K, max_pos, max_blocks, num_pages, page_size, splits, stages, nch, box_rows;
};

__device__ __forceinline__ void ld_ldsm4(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ld_ldsm4_t(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ld_ldsm2_t(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void ld_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// byte offset of 16-byte chunk c of row r in a tile kept as 64-element column blocks of [rows][128 bytes], 128-byte swizzle
__device__ __forceinline__ uint32_t ld_off(int r, int c, int rows) {
  return (uint32_t)((c >> 3) * rows * 128 + r * 128 + (((c & 7) ^ (r & 7)) << 4));
}
__device__ __forceinline__ void ld_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
__device__ __forceinline__ void ld_cluster_sync() {
  asm volatile("barrier.cluster.arrive.release;\n\tbarrier.cluster.wait.acquire;" ::: "memory");
}
__device__ __forceinline__ uint32_t ld_map(uint32_t addr, uint32_t rank) {   // shared address of another CTA of the cluster
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
  return r;
}
__device__ __forceinline__ float ld_remote_f(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ float4 ld_remote_f4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
  return v;
}

// MT: 16-head tiles per CTA; NT: 8-column tiles of O per warp (64 * NT >= kv_rank); BN: tokens per tile
template <int MT, int NT, int BN>
__global__ void __launch_bounds__(LD_THREADS, 1) attn_latent_decode_kernel(const __grid_constant__ CUtensorMap tmC, const LatentDecodeParams p) {
  constexpr int ROWS = 16 * MT;
  constexpr int NB = BN / 8;                       // 8-token units of a tile
  constexpr int MPW = MT * NB / LD_WARPS;          // head tiles per warp in the S phase
  constexpr int P_LD = BN + 8;                     // elements per row of P (16 bytes of padding: conflict-free ldmatrix)
  constexpr int S_LD = BN + 4;
  static_assert(MPW >= 1 && MPW * LD_WARPS == MT * NB, "tile shape");
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t bar_full[LD_MAX_STAGES], bar_empty[LD_MAX_STAGES];
  __shared__ float alpha_s[ROWS], m_s[ROWS], l_s[ROWS];
  __shared__ int abort_flag;
  pdl_trigger();
  pdl_wait();
  const int split = blockIdx.x, h0 = blockIdx.y * ROWS, t = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int K = p.K, nch = p.nch;
  int pos = p.positions[t];
  if (pos >= p.max_pos) { if (tid == 0) report_status(p.status, ST_BAD_INDEX, pos); pos = -1; }
  if (pos < 0) {      // padding row: the same decision in every CTA of the cluster
    if (split == 0)
      for (int i = tid; i < ROWS * K; i += LD_THREADS)
        if (h0 + i / K < p.H) p.out[(size_t)t * p.H * K + (size_t)h0 * K + i] = __float2bfloat16(0.f);
    return;
  }
  const int len = pos + 1, seq = p.seq_of_token ? p.seq_of_token[t] : t;
  const int n_all = (len + BN - 1) / BN, per = (n_all + p.splits - 1) / p.splits;
  const int tile0 = split * per;
  const int n_my = max(0, min(n_all - tile0, per));

  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
  const uint32_t stage_bytes = nch * BN * 128;
  const uint32_t q_s = base + p.stages * stage_bytes, p_s = q_s + nch * ROWS * 128;
  uint8_t* q_ptr = base_ptr + (q_s - base);
  __nv_bfloat16* p_ptr = reinterpret_cast<__nv_bfloat16*>(base_ptr + (p_s - base));
  float* s_ptr = reinterpret_cast<float*>(base_ptr + (p_s - base) + ROWS * P_LD * 2);

  if (tid == 0) {
    abort_flag = 0;
    for (int s = 0; s < p.stages; ++s) { mbar_init(smem_u32(&bar_full[s]), 1); mbar_init(smem_u32(&bar_empty[s]), LD_WARPS); }
    fence_mbar_init();
  }
  __syncthreads();

  float o[MT][NT][4];
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int b = 0; b < NT; ++b) o[a][b][0] = o[a][b][1] = o[a][b][2] = o[a][b][3] = 0.f;

  if (warp == LD_WARPS) {
    // ---------------------------------------------------------------- producer
    if (lane == 0) {
      tma_prefetch_desc(&tmC);
      const uint64_t pol = l2_policy_evict_first();
      const int* bt = p.block_table + (size_t)seq * p.max_blocks;
      const int ps = p.page_size, last_page = (len - 1) / ps;
      bool ok = true;
      int armed = 0;
      for (int j = 0; j < n_my; ++j) {
        const int s = j % p.stages;
        if (j >= p.stages && !mbar_wait(smem_u32(&bar_empty[s]), ((j / p.stages) - 1) & 1, &abort_flag, LD_BUDGET_NS)) { ok = false; break; }
        mbar_expect_tx(smem_u32(&bar_full[s]), stage_bytes);
        armed = j + 1;
        const uint32_t dst = base + s * stage_bytes;
        for (int r = 0; r < BN; r += p.box_rows) {
          const int tok = (tile0 + j) * BN + r;
          // a box past the end of the sequence repeats its last page: every row of the tile then holds finite values
          const int blk = min(tok / ps, last_page);
          int page = bt[blk];
          if (page < 0 || page >= p.num_pages) { report_status(p.status, ST_BAD_INDEX, page); page = 0; }
          const int row = page * ps + tok % ps;
          for (int c = 0; c < nch; ++c) tma_load_2d(dst + c * BN * 128 + r * 128, &tmC, smem_u32(&bar_full[s]), c * 64, row, pol);
        }
      }
      if (!ok) {
        abort_flag = 1;
        report_status(p.status, ST_TIMEOUT_SMEM_EMPTY, 30);
        volatile int never = 0;      // copies in flight still write this CTA's shared memory: wait for them (bounded)
        for (int j = max(0, armed - p.stages); j < armed; ++j)
          mbar_wait(smem_u32(&bar_full[j % p.stages]), (j / p.stages) & 1, &never, LD_BUDGET_NS);
      }
    }
  } else {
    // ---------------------------------------------------------------- queries -> shared memory (rows past H are zero)
    for (int i = tid; i < ROWS * nch * 8; i += LD_WARPS * 32) {
      const int r = i / (nch * 8), c = i % (nch * 8), col = c * 8, h = h0 + r;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (h < p.H && col < K) {
        v = *reinterpret_cast<const uint4*>(p.q_abs + (size_t)t * p.H * K + (size_t)h * K + col);
      } else if (h < p.H && col < K + p.rot) {
        const __nv_bfloat16* qr = p.q + (size_t)t * p.q_ld + (size_t)h * (p.D + p.rot) + p.D + (col - K);
        const float2* cs = reinterpret_cast<const float2*>(p.cos_sin) + (size_t)pos * (p.rot / 2) + (col - K) / 2;
        __nv_bfloat162* vb = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float u = __bfloat162float(qr[2 * k]), w = __bfloat162float(qr[2 * k + 1]);
          const float2 a = cs[k];
          vb[k] = __floats2bfloat162_rn(u * a.x - w * a.y, w * a.x + u * a.y);
        }
      }
      *reinterpret_cast<uint4*>(q_ptr + ld_off(r, c, ROWS)) = v;
    }
    float m_r[2 * MT], l_r[2 * MT];      // running maximum and sum of this warp's head rows warp * 2 MT .. (all lanes alike)
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i) { m_r[i] = -INFINITY; l_r[i] = 0.f; }
    ld_sync();
    const int nb = warp % NB, mg = warp / NB;      // S phase: 8-token unit, group of head tiles
    const int mat = lane >> 3;
    for (int j = 0; j < n_my; ++j) {
      const int s = j % p.stages;
      const uint32_t c_s = base + s * stage_bytes;
      const bool landed = mbar_wait(smem_u32(&bar_full[s]), (j / p.stages) & 1, &abort_flag, LD_BUDGET_NS);
      if (!landed) { report_status(p.status, ST_TIMEOUT_SMEM_FULL, 31); abort_flag = 1; }   // carries on: no barrier below is skipped
      // ---- S = Q C^T ----
      float sa[MPW][2][4];
#pragma unroll
      for (int a = 0; a < MPW; ++a)
#pragma unroll
        for (int b = 0; b < 2; ++b) sa[a][b][0] = sa[a][b][1] = sa[a][b][2] = sa[a][b][3] = 0.f;
      for (int k = 0; k < nch * 4; k += 2) {       // two 16-element steps at a time (columns past kv_rank + rot are zero)
        uint32_t b[4];
        ld_ldsm4(c_s + ld_off(nb * 8 + (lane & 7), k * 2 + mat, BN), b);
#pragma unroll
        for (int a = 0; a < MPW; ++a) {
          uint32_t q0[4], q1[4];
          const int row = (mg * MPW + a) * 16 + (lane & 15);
          ld_ldsm4(q_s + ld_off(row, k * 2 + (lane >> 4), ROWS), q0);
          ld_ldsm4(q_s + ld_off(row, k * 2 + 2 + (lane >> 4), ROWS), q1);
          ld_mma(sa[a][0], q0, b[0], b[1]);
          ld_mma(sa[a][1], q1, b[2], b[3]);
        }
      }
#pragma unroll
      for (int a = 0; a < MPW; ++a) {
        const int r = (mg * MPW + a) * 16 + (lane >> 2), c = nb * 8 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(s_ptr + r * S_LD + c) = make_float2(sa[a][0][0] + sa[a][1][0], sa[a][0][1] + sa[a][1][1]);
        *reinterpret_cast<float2*>(s_ptr + (r + 8) * S_LD + c) = make_float2(sa[a][0][2] + sa[a][1][2], sa[a][0][3] + sa[a][1][3]);
      }
      ld_sync();
      // ---- softmax of this warp's head rows ----
      const int valid = len - (tile0 + j) * BN;     // columns of the tile that exist (at least one)
#pragma unroll
      for (int i = 0; i < 2 * MT; ++i) {
        const int r = warp * 2 * MT + i;
        float x[BN / 32], mx = -INFINITY;
#pragma unroll
        for (int c = 0; c < BN / 32; ++c) {
          const int col = c * 32 + lane;
          x[c] = col < valid ? s_ptr[r * S_LD + col] * p.scale_log2e : -INFINITY;
          mx = fmaxf(mx, x[c]);
        }
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
        const float mn = fmaxf(m_r[i], mx), al = m_r[i] == -INFINITY ? 0.f : exp2f(m_r[i] - mn);
        float sum = 0.f;
#pragma unroll
        for (int c = 0; c < BN / 32; ++c) {
          const __nv_bfloat16 pb = __float2bfloat16(exp2f(x[c] - mn));
          sum += __bfloat162float(pb);
          p_ptr[r * P_LD + c * 32 + lane] = pb;
        }
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
        l_r[i] = l_r[i] * al + sum;
        m_r[i] = mn;
        if (lane == 0) alpha_s[r] = al;
      }
      ld_sync();
      // ---- O = alpha O + P C ----
#pragma unroll
      for (int a = 0; a < MT; ++a) {
        const float al0 = alpha_s[a * 16 + (lane >> 2)], al1 = alpha_s[a * 16 + (lane >> 2) + 8];
        if (__any_sync(0xffffffffu, al0 != 1.f || al1 != 1.f)) {
#pragma unroll
          for (int b = 0; b < NT; ++b) { o[a][b][0] *= al0; o[a][b][1] *= al0; o[a][b][2] *= al1; o[a][b][3] *= al1; }
        }
      }
#pragma unroll
      for (int k = 0; k < BN / 16; ++k) {
        uint32_t pf[MT][4];
#pragma unroll
        for (int a = 0; a < MT; ++a) ld_ldsm4(p_s + ((a * 16 + (lane & 15)) * P_LD + k * 16 + (lane >> 4) * 8) * 2, pf[a]);
        const int tok = k * 16 + (mat & 1) * 8 + (lane & 7);
        if (NT == 1) {
          if (warp * 8 < K) {
            uint32_t b[2];
            ld_ldsm2_t(c_s + ld_off(tok, warp, BN), b);       // lanes 0..15 give the addresses
#pragma unroll
            for (int a = 0; a < MT; ++a) ld_mma(o[a][0], pf[a], b[0], b[1]);
          }
        } else {
#pragma unroll
          for (int n = 0; n < NT; n += 2) {
            if ((warp * NT + n) * 8 < K) {
              uint32_t b[4];
              ld_ldsm4_t(c_s + ld_off(tok, warp * NT + n + (mat >> 1), BN), b);
#pragma unroll
              for (int a = 0; a < MT; ++a) {
                ld_mma(o[a][n], pf[a], b[0], b[1]);
                ld_mma(o[a][NT > 1 ? n + 1 : 0], pf[a], b[2], b[3]);
              }
            }
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&bar_empty[s]));
    }
    if (lane == 0) {
#pragma unroll
      for (int i = 0; i < 2 * MT; ++i) { m_s[warp * 2 * MT + i] = m_r[i]; l_s[warp * 2 * MT + i] = l_r[i]; }
    }
    ld_sync();       // every warp is done with the ring: its memory becomes the parking place of O, [ROWS][K] fp32
    float* park = reinterpret_cast<float*>(base_ptr);
#pragma unroll
    for (int a = 0; a < MT; ++a)
#pragma unroll
      for (int b = 0; b < NT; ++b) {
        const int col = (warp * NT + b) * 8 + (lane & 3) * 2, r = a * 16 + (lane >> 2);
        if (col < K) {
          *reinterpret_cast<float2*>(park + (size_t)r * K + col) = make_float2(o[a][b][0], o[a][b][1]);
          *reinterpret_cast<float2*>(park + (size_t)(r + 8) * K + col) = make_float2(o[a][b][2], o[a][b][3]);
        }
      }
  }
  // ---- merge: CTA `split` of the cluster produces every splits-th head row of the group ----
  const int ns = p.splits;
  if (ns > 1) ld_cluster_sync(); else __syncthreads();
  const uint32_t m_a = smem_u32(m_s), l_a = smem_u32(l_s);
  const int q4 = K / 4, n_rows = (ROWS - split + ns - 1) / ns;
  for (int i = tid; i < n_rows * q4; i += LD_THREADS) {
    const int r = split + (i / q4) * ns, col = (i % q4) * 4;
    if (h0 + r >= p.H) continue;
    float M = -INFINITY;
    for (int c = 0; c < ns; ++c) M = fmaxf(M, ns > 1 ? ld_remote_f(ld_map(m_a + r * 4, c)) : m_s[r]);
    float L = 0.f;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int c = 0; c < ns; ++c) {
      const float mc = ns > 1 ? ld_remote_f(ld_map(m_a + r * 4, c)) : m_s[r];
      const float lc = ns > 1 ? ld_remote_f(ld_map(l_a + r * 4, c)) : l_s[r];
      const float w = mc == -INFINITY ? 0.f : exp2f(mc - M);
      const uint32_t oa = base + (uint32_t)(((size_t)r * K + col) * 4);
      const float4 v = ns > 1 ? ld_remote_f4(ld_map(oa, c)) : *reinterpret_cast<const float4*>(base_ptr + ((size_t)r * K + col) * 4);
      L += w * lc;
      acc.x += w * v.x; acc.y += w * v.y; acc.z += w * v.z; acc.w += w * v.w;
    }
    const float inv = L > 0.f ? 1.f / L : 0.f;
    const __nv_bfloat162 a = __floats2bfloat162_rn(acc.x * inv, acc.y * inv), b = __floats2bfloat162_rn(acc.z * inv, acc.w * inv);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&a); u.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p.out + (size_t)t * p.H * K + (size_t)(h0 + r) * K + col) = u;
  }
  if (ns > 1) ld_cluster_sync();      // nobody leaves while another CTA reads its shared memory
}

template <int MT, int NT, int BN>
static int latent_decode_launch(const CUtensorMap& tm, LatentDecodeParams& p, int T, int groups, cudaStream_t s) {
  constexpr int ROWS = 16 * MT;
  const int stage = p.nch * BN * 128;
  const int fixed = p.nch * ROWS * 128 + ROWS * (BN + 8) * 2 + ROWS * (BN + 4) * 4 + 1024 + 64;
  int st = (220 * 1024 - fixed) / stage;
  if (st > LD_MAX_STAGES) st = LD_MAX_STAGES;
  if (st < 2) return -1;
  p.stages = st;
  size_t smem = (size_t)st * stage + fixed;
  const size_t park = (size_t)ROWS * p.K * 4 + 1024;
  if (park > smem) smem = park;
  auto fn = attn_latent_decode_kernel<MT, NT, BN>;
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
// multiples of 16, kv_rank <= 512, page sizes 16, 32 or a multiple of 64. splits 0: chosen from the row count and ctx_hint.
extern "C" int skein_latent_attn_decode(const void* q_abs, const void* q, long long q_ld, const float* cos_sin, int max_pos,
                                        const int* positions, const int* seq_of_token, const int* block_table, int max_blocks,
                                        const void* cache, int num_pages, int page_size, void* out, int T, int H, int D, int rot, int kv_rank,
                                        float scale, int splits, int ctx_hint, int* status, void* stream) {
  using namespace skein;
  if (T == 0) return 0;
  if (kv_rank % 16 || rot % 16 || kv_rank < 16 || kv_rank > 512 || rot < 16 || T > 65535 || scale <= 0.f) return -1;
  if (!(page_size == 16 || page_size == 32 || page_size % 64 == 0)) return -1;
  LatentDecodeParams p;
  p.q_abs = (const __nv_bfloat16*)q_abs; p.q = (const __nv_bfloat16*)q; p.cos_sin = cos_sin; p.positions = positions;
  p.seq_of_token = seq_of_token; p.block_table = block_table; p.out = (__nv_bfloat16*)out; p.status = status; p.q_ld = q_ld;
  p.scale_log2e = scale * 1.4426950408889634f;
  p.H = H; p.D = D; p.rot = rot; p.K = kv_rank; p.max_pos = max_pos; p.max_blocks = max_blocks; p.num_pages = num_pages; p.page_size = page_size;
  p.nch = (kv_rank + rot + 63) / 64;
  const int mt = H <= 16 ? 1 : H <= 32 ? 2 : 4, bn = mt == 4 ? 32 : 64;
  const int groups = (H + 16 * mt - 1) / (16 * mt);
  p.box_rows = page_size < bn ? page_size : bn;
  int dev = 0, sms = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms <= 0) sms = 148;
  if (splits <= 0) {
    splits = sms / (T * groups > 0 ? T * groups : 1);
    if (splits > ctx_hint / bn) splits = ctx_hint / bn;
  }
  p.splits = splits < 1 ? 1 : splits > LD_MAX_SPLITS ? LD_MAX_SPLITS : splits;
  CUtensorMap tm;
  const int rc = cached_tmap_2d(&tm, cache, (uint64_t)num_pages * page_size, (uint64_t)(kv_rank + rot), 2, p.box_rows);
  if (rc != 0) return rc;
  const int nt = kv_rank <= 64 ? 1 : kv_rank <= 128 ? 2 : kv_rank <= 256 ? 4 : 8;
  cudaStream_t s = (cudaStream_t)stream;
#define LD_CASE(M, N, B) if (mt == M && nt == N) return latent_decode_launch<M, N, B>(tm, p, T, groups, s);
  LD_CASE(1, 1, 64) LD_CASE(1, 2, 64) LD_CASE(1, 4, 64) LD_CASE(1, 8, 64)
  LD_CASE(2, 1, 64) LD_CASE(2, 2, 64) LD_CASE(2, 4, 64) LD_CASE(2, 8, 64)
  LD_CASE(4, 1, 32) LD_CASE(4, 2, 32) LD_CASE(4, 4, 32) LD_CASE(4, 8, 32)
#undef LD_CASE
  return -1;
}
