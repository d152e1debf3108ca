// Expert selection and the expert-sorted layout of a decode step, shared by the kernels that fuse the MoE router into the
// norm before it (norm.cu: pre-norm blocks, postnorm.cu: post-norm blocks).
#pragma once
#include "ptx.cuh"
#include <cuda_bf16.h>
#include <math.h>
#include <stdint.h>

// Rule of a group-limited choice of experts (mirrored in skein_b200/ops/_lib.py).
extern "C" typedef struct SkeinRouteRule {
  int32_t n_groups, keep;    // equal groups of neighbours, of which the best `keep` are eligible
  int32_t score;             // ROUTE_*
  int32_t group_best;        // a group's score is the sum of its 1 or 2 best
  int32_t renorm;            // the chosen scores are divided by their sum
  float scale;               // ... and multiplied by this
} SkeinRouteRule;

namespace skein {

enum : int { ROUTE_SOFTMAX = 0, ROUTE_SIGMOID = 1 };
inline bool route_rule_ok(const SkeinRouteRule& r, int E, int topk) {
  return r.n_groups >= 1 && r.n_groups <= 64 && E % r.n_groups == 0 && r.keep >= 1 && r.keep <= r.n_groups && topk >= 1 && topk <= r.keep * (E / r.n_groups) &&
         r.group_best >= 1 && r.group_best <= 2;
}

constexpr int NR_MAX_E = 64;
constexpr int NR_MAX_K = 8;
constexpr int NR_MAX_PAIRS = 2048;

struct RouteParams {
  const __nv_bfloat16* wg;   // [E, H]
  int* expert_ids;           // [T, k]
  float* expert_w;           // [T, k]
  int* counts;               // [E]
  int* offsets;              // [E + 1]
  int* row_of;               // [T * k]   (-1: expert not on this rank)
  int* src_token;            // [T * k]
  __nv_bfloat16* xs;         // [T * k, H] rows in expert-sorted order
  int* barrier;              // [2] arrive / depart, zero between launches
  int E, topk, e_first, e_count;
  unsigned long long barrier_budget_ns;
};

struct RouteShared {
  float part[16][NR_MAX_E];
  float logit[NR_MAX_E];
  int ids[NR_MAX_PAIRS];
  int cnt[NR_MAX_E], bef[NR_MAX_E], off[NR_MAX_E + 1];
  int my_row[NR_MAX_K];
  int barrier_ok;
};

// logits of this CTA's row against all experts from the row's bf16 values held in registers (thread tid owns elements
// ps * blockDim * 8 + tid * 8 ..): per-warp partial sums in s.part. Needs a barrier before route_sum_logits.
template <int MAX_PASSES>
__device__ __forceinline__ void route_partial_logits(const uint4 (&nb)[MAX_PASSES], bool have_row, const __nv_bfloat16* wg, int E, int H,
                                                     RouteShared& s) {
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int per_pass = blockDim.x * 8;
  for (int e0 = 0; e0 < E; e0 += 8) {
    float a[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) a[i] = 0.f;
    if (have_row) {
#pragma unroll
      for (int ps = 0; ps < MAX_PASSES; ++ps) {
        const int h = ps * per_pass + tid * 8;
        if (h >= H) break;
        uint4 wr[8];
#pragma unroll
        for (int i = 0; i < 8; ++i)
          wr[i] = (e0 + i < E) ? *reinterpret_cast<const uint4*>(wg + (size_t)(e0 + i) * H + h) : make_uint4(0, 0, 0, 0);
        const __nv_bfloat162* xb = reinterpret_cast<const __nv_bfloat162*>(&nb[ps]);
        float xf[8];
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(xb[i]); xf[2 * i] = f.x; xf[2 * i + 1] = f.y; }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const __nv_bfloat162* wb = reinterpret_cast<const __nv_bfloat162*>(&wr[i]);
#pragma unroll
          for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(wb[j]); a[i] += xf[2 * j] * f.x + xf[2 * j + 1] * f.y; }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      float v = a[i];
      for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      if (lane == 0 && e0 + i < E) s.part[warp][e0 + i] = v;
    }
  }
}

__device__ __forceinline__ float route_sum_logit(const RouteShared& s, int e) {
  float v = 0.f;
  const int nwarps = blockDim.x >> 5;
  for (int w = 0; w < nwarps; ++w) v += s.part[w][e];
  return v;
}

// One thread, after it stored this row's expert ids and weights: publish them and wait (bounded) until every row has.
__device__ __forceinline__ void route_publish_and_wait(const RouteParams& r, int* status, int t, int T, RouteShared& s) {
  // release at device scope: this thread's stores of the expert ids / weights above are visible to whoever acquires
  // the counter (one instruction instead of a full fence followed by a relaxed add)
  asm volatile("red.release.gpu.global.add.s32 [%0], 1;" ::"l"(r.barrier) : "memory");
  // grid-wide arrival, bounded: all T CTAs are resident, so this only runs out if one never started
  const bool poisoned = status != nullptr && *(volatile int*)status == ST_TIMEOUT_GRID_BARRIER;
  const bool ok = !poisoned && wait_counter_ge_gpu(r.barrier, T, r.barrier_budget_ns);
  if (!ok) report_status(status, ST_TIMEOUT_GRID_BARRIER, t);
  s.barrier_ok = ok ? 1 : 0;
}

// Every CTA, after a barrier behind route_publish_and_wait: derives the expert-sorted layout (counts, exclusive offsets;
// pair (t, j) sits at offsets[e] + number of earlier pairs routed to e) and writes its own row to xs for its k experts.
template <int MAX_PASSES>
__device__ __forceinline__ void route_scatter(const RouteParams& r, const uint4 (&nb)[MAX_PASSES], bool have_row, int H, int t, int T,
                                              RouteShared& s) {
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nwarps = blockDim.x >> 5;
  const int E = r.E, topk = r.topk, per_pass = blockDim.x * 8;
  const int n_pairs = T * topk;
  for (int i = tid; i < n_pairs; i += blockDim.x) s.ids[i] = __ldcg(r.expert_ids + i);
  __syncthreads();
  const int my_first = t * topk;
  for (int e = warp; e < E; e += nwarps) {
    int c = 0, before = 0;
    for (int i0 = 0; i0 < n_pairs; i0 += 32) {
      const int i = i0 + lane;
      const bool hit = i < n_pairs && s.ids[i] == e;
      c += __popc(__ballot_sync(0xffffffffu, hit));
      before += __popc(__ballot_sync(0xffffffffu, hit && i < my_first));
    }
    if (lane == 0) {
      s.cnt[e] = (e >= r.e_first && e < r.e_first + r.e_count) ? c : 0;
      s.bef[e] = before;
    }
  }
  __syncthreads();
  if (tid == 0) {
    int a = 0;
    for (int e = 0; e < E; ++e) { s.off[e] = a; a += s.cnt[e]; }
    s.off[E] = a;
    if (t == 0) {
      for (int e = 0; e < E; ++e) { r.counts[e] = s.cnt[e]; r.offsets[e] = s.off[e]; }
      r.offsets[E] = a;
    }
    for (int j = 0; j < topk; ++j) {
      const int e = s.ids[my_first + j];
      const bool mine = e >= r.e_first && e < r.e_first + r.e_count;
      const int row = mine ? s.off[e] + s.bef[e] : -1;   // a token's k experts are distinct
      s.my_row[j] = row;
      r.row_of[my_first + j] = row;
      if (row >= 0) r.src_token[row] = t;
    }
  }
  __syncthreads();
  if (have_row && r.xs != nullptr) {
#pragma unroll
    for (int ps = 0; ps < MAX_PASSES; ++ps) {
      const int h = ps * per_pass + tid * 8;
      if (h >= H) break;
      for (int j = 0; j < topk; ++j) {
        const int row = s.my_row[j];
        if (row >= 0) *reinterpret_cast<uint4*>(r.xs + (size_t)row * H + h) = nb[ps];
      }
    }
  }
  if (tid == 0) {
    const int old = atomicAdd(r.barrier + 1, 1);
    if (old == T - 1) { r.barrier[0] = 0; r.barrier[1] = 0; }   // every CTA is past the wait: re-arm
  }
}

// Group-limited selection by one warp over the logits z of E experts (shared memory): a score per expert, experts in n_groups equal groups
// of neighbours of which the `keep` best are eligible (a group counts its best or its two best scores), the topk best eligible experts in
// descending order (ties to the lower index), their scores as weights, divided by their sum with renorm, times scale. Lane 0 writes ids / w
// (shared or global memory).
__device__ __forceinline__ void warp_argmax(float& v, int& i) {
  for (int o = 16; o > 0; o >>= 1) {
    const float v2 = __shfl_xor_sync(0xffffffffu, v, o);
    const int i2 = __shfl_xor_sync(0xffffffffu, i, o);
    if (v2 > v || (v2 == v && i2 < i)) { v = v2; i = i2; }
  }
}
__device__ __forceinline__ float warp_sum(float v) {
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
template <int MAX_E>
__device__ __forceinline__ void select_grouped_warp(const float* z, int E, int topk, const SkeinRouteRule& rule, int* ids, float* w) {
  constexpr int PER = (MAX_E + 31) / 32;
  const int lane = threadIdx.x & 31;
  // v: what is compared. Softmax scores rise with the logits, so there the logits themselves are compared.
  float v[PER];
  float mx = -INFINITY, den = 0.f;
#pragma unroll
  for (int q = 0; q < PER; ++q) {
    const int e = q * 32 + lane;
    // a logit that is not a number counts as the smallest: the indices below stay valid whatever the input
    v[q] = (e < E && z[e] == z[e]) ? fmaxf(z[e], -3.0e38f) : (e < E ? -3.0e38f : -INFINITY);
    if (rule.score == ROUTE_SIGMOID && e < E) v[q] = 1.f / (1.f + expf(-v[q]));
    mx = fmaxf(mx, v[q]);
  }
  if (rule.score == ROUTE_SOFTMAX) {
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
#pragma unroll
    for (int q = 0; q < PER; ++q) if (q * 32 + lane < E) den += expf(v[q] - mx);
    den = warp_sum(den);
  }
  if (rule.keep < rule.n_groups) {
    const int per = E / rule.n_groups;
    unsigned long long kept = 0;     // at most 64 groups
    if (rule.group_best > 1) {
      // lane g owns groups g and g + 32; the members' scores come from the lanes that hold them
      float worth[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        if (h * 32 >= rule.n_groups) break;
        const int g = h * 32 + lane;
        float b1 = -INFINITY, b2 = -INFINITY;
        for (int i = 0; i < per; ++i) {
          const int e = g < rule.n_groups ? g * per + i : 0;
          float s = 0.f;
#pragma unroll
          for (int q = 0; q < PER; ++q) {
            const float c = __shfl_sync(0xffffffffu, v[q], e & 31);
            if ((e >> 5) == q) s = c;
          }
          if (rule.score == ROUTE_SOFTMAX) s = expf(s - mx);
          if (s > b1) { b2 = b1; b1 = s; }
          else if (s > b2) b2 = s;
        }
        if (g < rule.n_groups) worth[h] = per > 1 ? b1 + b2 : b1;
      }
      for (int k = 0; k < rule.keep; ++k) {
        float bv = -INFINITY;
        int bi = 64;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int g = h * 32 + lane;
          if (g < rule.n_groups && !((kept >> g) & 1ull) && (worth[h] > bv || bi == 64)) { bv = worth[h]; bi = g; }
        }
        warp_argmax(bv, bi);
        if (bi < 64) kept |= 1ull << bi;
      }
    } else {
      for (int k = 0; k < rule.keep; ++k) {
        float bv = -INFINITY;
        int bi = MAX_E;
#pragma unroll
        for (int q = 0; q < PER; ++q) {
          const int e = q * 32 + lane;
          if (e < E && !((kept >> (e / per)) & 1ull) && (v[q] > bv || bi == MAX_E)) { bv = v[q]; bi = e; }
        }
        warp_argmax(bv, bi);
        if (bi < MAX_E) kept |= 1ull << (bi / per);
      }
    }
#pragma unroll
    for (int q = 0; q < PER; ++q) {
      const int e = q * 32 + lane;
      if (e < E && !((kept >> (e / per)) & 1ull)) v[q] = -INFINITY;
    }
  }
  float sum = 0.f;
  for (int j = 0; j < topk; ++j) {
    float bv = -INFINITY;
    int bi = MAX_E;
#pragma unroll
    for (int q = 0; q < PER; ++q) {
      const int e = q * 32 + lane;
      if (v[q] > -INFINITY && (v[q] > bv || bi == MAX_E)) { bv = v[q]; bi = e; }
    }
    warp_argmax(bv, bi);
    const float s = bi >= E ? 0.f : rule.score == ROUTE_SIGMOID ? bv : expf(bv - mx) / den;
    sum += s;
    if (lane == 0) { ids[j] = bi < E ? bi : 0; w[j] = s * rule.scale; }
#pragma unroll
    for (int q = 0; q < PER; ++q) if (q * 32 + lane == bi) v[q] = -INFINITY;
  }
  if (rule.renorm) {
    __syncwarp();
    if (lane == 0) for (int j = 0; j < topk; ++j) w[j] = w[j] / (sum + 1e-20f);
  }
}

}  // namespace skein
