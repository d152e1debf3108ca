// Kernels between the products of a pre-norm layer whose stream x is fp32:
//
//   add_norm     a = x + sum_j w_j y[row_j] + step (each optional), fp32;  act = a / sqrt(mean(a^2) + eps) * gain
//   depth_norm   a = sum_j w_j X_j over the embedding output and the results of the layers so far, fp32;  h = a / rms(a) * gain with a root mean
//                square per group of neighbouring elements;  act = h + (h of the previous token - h) * shift. A sequence's last h is kept
//                in its state slot
//   norm_route   add_norm's norm of x for decode-sized bf16 steps, followed in the same launch by the router and the scatter of the row
//                into expert-sorted order (route.cuh)
//
// T is the activation type (bf16, or fp32 when a model runs in 32-bit); everything between the loads and the stores is fp32.
#include "ptx.cuh"
#include "launch.cuh"
#include "route.cuh"
#include "vec.cuh"
#include <cuda_bf16.h>
#include <math.h>

namespace skein {

struct AddNormParams {
  const float* x;            // [B, C]
  const void* y;             // [rows, C] activation type, or null
  const int* row_idx;        // [B, topk] rows of y
  const float* row_w;        // [B, topk] weights
  const float* step;         // [C] or null
  const float* gain;         // [C] or null (no norm)
  float* x_out;              // [B, C] or null
  void* act_out;             // [B, C] activation type, or null
  float eps;
  int C, topk;
};

__device__ __forceinline__ float nr_block_sum(float v, float* sh) {
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (l == 0) sh[w] = v;
  __syncthreads();
  float t = (l < nw) ? sh[l] : 0.f;
  for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
  return t;
}

// V elements of the sum at column i of row b
template <typename T, int V>
__device__ __forceinline__ void add_sum(const AddNormParams& p, int b, int i, float* a) {
  load_v<float, V>(p.x + (size_t)b * p.C + i, a);
  if (p.step) {
    float s[V];
    load_v<float, V>(p.step + i, s);
#pragma unroll
    for (int k = 0; k < V; ++k) a[k] += s[k];
  }
  if (p.y == nullptr) return;
  for (int j0 = 0; j0 < p.topk; j0 += 8) {       // rows in batches of 8: all loads of a batch are issued before the first is used
    float v[8][V], w8[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      w8[j] = 0.f;
      if (j0 + j < p.topk) {
        const int row = p.row_idx[(size_t)b * p.topk + j0 + j];
        w8[j] = row < 0 ? 0.f : p.row_w[(size_t)b * p.topk + j0 + j];
        load_v<T, V>((const T*)p.y + (size_t)(row < 0 ? 0 : row) * p.C + i, v[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (j0 + j < p.topk)
#pragma unroll
        for (int k = 0; k < V; ++k) a[k] = fmaf(w8[j], v[j][k], a[k]);
  }
}

// One CTA per row. PASSES: V elements per thread and pass stay in registers; 0: any row length, parked in dynamic shared memory.
template <typename T, int V, int PASSES>
__global__ void __launch_bounds__(PASSES >= 4 ? 512 : 1024) add_norm_kernel(const AddNormParams p) {
  extern __shared__ __align__(16) float row_sm[];
  __shared__ float sh[32];
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x, tid = threadIdx.x, hop = blockDim.x * V;
  float vals[PASSES > 0 ? PASSES : 1][V];
  float ss = 0.f;
  auto take = [&](int i, float* a) {
    add_sum<T, V>(p, b, i, a);
    if (p.x_out) store_v<float, V>(p.x_out + (size_t)b * p.C + i, a);
#pragma unroll
    for (int k = 0; k < V; ++k) ss = fmaf(a[k], a[k], ss);
  };
  if (PASSES > 0) {
#pragma unroll
    for (int ps = 0; ps < (PASSES > 0 ? PASSES : 1); ++ps)
      if (ps * hop + tid * V < p.C) take(ps * hop + tid * V, vals[ps]);
  } else {
    for (int i = tid * V; i < p.C; i += hop) {
      float a[V];
      take(i, a);
#pragma unroll
      for (int k = 0; k < V; ++k) row_sm[i + k] = a[k];
    }
  }
  if (p.act_out == nullptr) return;
  const float r = 1.f / sqrtf(nr_block_sum(ss, sh) / (float)p.C + p.eps);
  auto put = [&](int i, const float* a) {
    float g[V];
    load_v<float, V>(p.gain + i, g);
#pragma unroll
    for (int k = 0; k < V; ++k) g[k] *= a[k] * r;
    store_v<T, V>((T*)p.act_out + (size_t)b * p.C + i, g);
  };
  if (PASSES > 0) {
#pragma unroll
    for (int ps = 0; ps < (PASSES > 0 ? PASSES : 1); ++ps)
      if (ps * hop + tid * V < p.C) put(ps * hop + tid * V, vals[ps]);
  } else {
    for (int i = tid * V; i < p.C; i += hop) put(i, row_sm + i);
  }
}

}  // namespace skein

// Mirrored in skein_b200/ops/_lib.py (keep the field order identical there).
extern "C" typedef struct SkeinDepthNormParams {
  const float* terms;            // [n_terms] matrices [T, C], term_stride elements apart
  const float* weights;          // [n_terms], or null (one term of weight 1)
  float* x_out;                  // [T, C] the sum, or null
  const float* gain;             // [C]
  void* act_out;                 // [T, C] activation type
  const float* shift;            // [C], or null: act is h. With it:
  float* state;                  // [num_slots, C] every sequence's last h
  const int32_t* positions;      // [T], -1: padding row; position 0 starts from zero whatever the slot holds
  const int32_t* slots;          // [sequences]
  const int32_t* seq_of_token;   // [T], or null: every row is the next token of its own sequence
  const int32_t* q_start;        // [sequences] first row of each portion
  const int32_t* q_len;
  int32_t* status;
  int64_t term_stride;
  int32_t n_terms, T, C, groups, num_slots;
  float eps;
} SkeinDepthNormParams;

namespace skein {

using DepthNormParams = SkeinDepthNormParams;
constexpr int DN_SEG = 128;            // elements that a warp holds per pass
constexpr int DN_MAX_SEGS = 64;

// V elements of the weighted sum at column i of row t
template <int V>
__device__ __forceinline__ void depth_sum(const DepthNormParams& p, int t, int i, float* a) {
  const float* x = p.terms + (size_t)t * p.C + i;
  if (p.weights == nullptr) { load_v<float, V>(x, a); return; }
#pragma unroll
  for (int k = 0; k < V; ++k) a[k] = 0.f;
  for (int j0 = 0; j0 < p.n_terms; j0 += 4) {      // four loads in flight
    float v[4][V], w[4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (j0 + j < p.n_terms) {
        w[j] = p.weights[j0 + j];
        load_v<float, V>(x + (size_t)(j0 + j) * p.term_stride, v[j]);
      }
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (j0 + j < p.n_terms)
#pragma unroll
        for (int k = 0; k < V; ++k) a[k] = fmaf(w[j], v[j][k], a[k]);
  }
}

// The rows [r0, r1) of a CTA in order, so that a row's h is at hand for the next one. row(t, store, dst) computes h of row t (store: its sum
// goes to x_out) into one of three buffers, put(t, shifted) writes act from buffers 0 (h) and 1 (h of the previous token) and moves 0 to 1;
// take(slot, zero) fills buffer 1 from the state, keep(slot, buffer) writes it. The CTA of a portion's first row also keeps the portion's
// last h, once it has read the old one, whichever CTA the last row belongs to.
template <typename Row, typename Put, typename Take, typename Keep>
__device__ __forceinline__ void depth_walk(const DepthNormParams& p, int r0, int r1, Row row, Put put, Take take, Keep keep) {
  for (int t = r0; t < r1; ++t) {
    row(t, true, 0);
    const int pos = p.shift ? p.positions[t] : -1;
    if (pos < 0) { put(t, false); continue; }
    const int seq = p.seq_of_token ? p.seq_of_token[t] : t, first = p.q_start ? p.q_start[seq] : t;
    if (t == first) {
      const int slot = p.slots[seq], len = p.q_len ? p.q_len[seq] : 1;
      if (slot < 0 || slot >= p.num_slots) { if (threadIdx.x == 0) report_status(p.status, ST_BAD_INDEX, slot); return; }
      take(slot, pos == 0);
      if (len > 1) row(first + len - 1, false, 2);
      keep(slot, len > 1 ? 2 : 0);
    } else if (t == r0) {
      row(t - 1, false, 1);
    }
    put(t, true);
  }
}

// A thread keeps 4 elements per pass in registers; groups of a multiple of DN_SEG elements, so that a warp's pass lies in one.
template <typename T, int PASSES, bool SHIFT>
__global__ void __launch_bounds__(512) depth_norm_kernel(const DepthNormParams p, int rows) {
  __shared__ float seg[2][DN_MAX_SEGS];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, hop = blockDim.x * 4, group = p.C / p.groups, per = group / DN_SEG;
  float b[3][PASSES][4];
  int flip = 0;
  auto each = [&](auto f) {
#pragma unroll
    for (int ps = 0; ps < PASSES; ++ps) {
      const int i = ps * hop + tid * 4;
      if (i < p.C) f(i, ps);
    }
  };
  auto row_into = [&](int t, bool store, float (&h)[PASSES][4]) {
    float* sh = seg[flip];           // two in turn: a warp can be one row ahead of another, not two
    flip ^= 1;
#pragma unroll
    for (int ps = 0; ps < PASSES; ++ps) {
      const int i = ps * hop + tid * 4;
      float ss = 0.f;
      if (i < p.C) {
        depth_sum<4>(p, t, i, h[ps]);
        if (store && p.x_out) store_v<float, 4>(p.x_out + (size_t)t * p.C + i, h[ps]);
        ss = h[ps][0] * h[ps][0] + h[ps][1] * h[ps][1] + h[ps][2] * h[ps][2] + h[ps][3] * h[ps][3];
      }
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (lane == 0 && ps * hop + warp * DN_SEG < p.C) sh[(ps * hop + warp * DN_SEG) / DN_SEG] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int ps = 0; ps < PASSES; ++ps) {
      const int i0 = ps * hop + warp * DN_SEG;
      if (i0 >= p.C) break;          // (the whole warp)
      const int g = i0 / group;
      float ss = 0.f;
      for (int j = lane; j < per; j += 32) ss += sh[g * per + j];
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float r = 1.f / sqrtf(ss / (float)group + p.eps);
      float w[4];
      load_v<float, 4>(p.gain + i0 + lane * 4, w);
#pragma unroll
      for (int k = 0; k < 4; ++k) h[ps][k] *= r * w[k];
    }
  };
  auto row = [&](int t, bool store, int to) {      // (`to` is a constant where this is inlined)
    if (to == 0) row_into(t, store, b[0]);
    else if (to == 1) row_into(t, store, b[1]);
    else row_into(t, store, b[2]);
  };
  auto put = [&](int t, bool shifted) {
    each([&](int i, int ps) {
      float o[4], m[4];
      if (shifted) {
        load_v<float, 4>(p.shift + i, m);
#pragma unroll
        for (int k = 0; k < 4; ++k) { o[k] = fmaf(b[1][ps][k] - b[0][ps][k], m[k], b[0][ps][k]); b[1][ps][k] = b[0][ps][k]; }
      }
      store_v<T, 4>((T*)p.act_out + (size_t)t * p.C + i, shifted ? o : b[0][ps]);
    });
  };
  auto take = [&](int slot, bool zero) {
    each([&](int i, int ps) {
      if (!zero) load_v<float, 4>(p.state + (size_t)slot * p.C + i, b[1][ps]);
      else b[1][ps][0] = b[1][ps][1] = b[1][ps][2] = b[1][ps][3] = 0.f;
    });
  };
  auto keep = [&](int slot, int from) {
    each([&](int i, int ps) { store_v<float, 4>(p.state + (size_t)slot * p.C + i, from == 2 ? b[2][ps] : b[0][ps]); });
  };
  const int r0 = blockIdx.x * rows, r1 = min(r0 + rows, p.T);
  if (SHIFT) depth_walk(p, r0, r1, row, put, take, keep);
  else for (int t = r0; t < r1; ++t) { row(t, true, 0); put(t, false); }
}

// Any row length and group size: the three buffers in shared memory, then a factor per group.
template <typename T>
__global__ void __launch_bounds__(512) depth_norm_any_kernel(const DepthNormParams p, int rows) {
  extern __shared__ __align__(16) float row_sm[];      // [3][C], [groups]
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, group = p.C / p.groups;
  float* fac = row_sm + 3 * p.C;
  auto row = [&](int t, bool store, int to) {
    float* h = row_sm + to * p.C;
    for (int i = tid; i < p.C; i += blockDim.x) {
      depth_sum<1>(p, t, i, h + i);
      if (store && p.x_out) p.x_out[(size_t)t * p.C + i] = h[i];
    }
    __syncthreads();
    for (int g = warp; g < p.groups; g += blockDim.x >> 5) {
      float ss = 0.f;
      for (int i = lane; i < group; i += 32) ss = fmaf(h[g * group + i], h[g * group + i], ss);
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (lane == 0) fac[g] = 1.f / sqrtf(ss / (float)group + p.eps);
    }
    __syncthreads();
    for (int i = tid; i < p.C; i += blockDim.x) h[i] *= fac[i / group] * p.gain[i];      // (from here on a thread reads what it wrote)
  };
  auto put = [&](int t, bool shifted) {
    for (int i = tid; i < p.C; i += blockDim.x) {
      const float h = row_sm[i];
      ((T*)p.act_out)[(size_t)t * p.C + i] = from_f<T>(shifted ? fmaf(row_sm[p.C + i] - h, p.shift[i], h) : h);
      row_sm[p.C + i] = h;
    }
  };
  auto take = [&](int slot, bool zero) {
    for (int i = tid; i < p.C; i += blockDim.x) row_sm[p.C + i] = zero ? 0.f : p.state[(size_t)slot * p.C + i];
  };
  auto keep = [&](int slot, int from) {
    for (int i = tid; i < p.C; i += blockDim.x) p.state[(size_t)slot * p.C + i] = row_sm[from * p.C + i];
  };
  const int r0 = blockIdx.x * rows;
  depth_walk(p, r0, min(r0 + rows, p.T), row, put, take, keep);
}

struct NormRouteParams {
  const float* x;            // [B, C]
  const float* gain;         // [C]
  __nv_bfloat16* act_out;    // [B, C]
  int* status;
  float eps;
  int C;
};

// One CTA per row, all resident at once; a thread owns 8 consecutive elements per pass.
template <int MAX_PASSES>
__global__ void __launch_bounds__(512) norm_route_kernel(const NormRouteParams p, const RouteParams r, const SkeinRouteRule rule) {
  __shared__ float sh[32];
  __shared__ RouteShared rs;
  __shared__ int sel_id[NR_MAX_K];
  __shared__ float sel_w[NR_MAX_K];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, T = gridDim.x;
  const int per_pass = blockDim.x * 8;
  float vals[MAX_PASSES][8], gain[MAX_PASSES][8];
  float ss = 0.f;
#pragma unroll
  for (int ps = 0; ps < MAX_PASSES; ++ps) {
    const int h = ps * per_pass + tid * 8;
    if (h >= p.C) break;
    load_v<float, 4>(p.x + (size_t)t * p.C + h, vals[ps]);
    load_v<float, 4>(p.x + (size_t)t * p.C + h + 4, vals[ps] + 4);
    load_v<float, 4>(p.gain + h, gain[ps]);
    load_v<float, 4>(p.gain + h + 4, gain[ps] + 4);
#pragma unroll
    for (int k = 0; k < 8; ++k) ss = fmaf(vals[ps][k], vals[ps][k], ss);
  }
  const float scale = 1.f / sqrtf(nr_block_sum(ss, sh) / (float)p.C + p.eps);
  uint4 nb[MAX_PASSES];
#pragma unroll
  for (int ps = 0; ps < MAX_PASSES; ++ps) {
    const int h = ps * per_pass + tid * 8;
    if (h >= p.C) break;
    __nv_bfloat162* ob = reinterpret_cast<__nv_bfloat162*>(&nb[ps]);
#pragma unroll
    for (int k = 0; k < 4; ++k)
      ob[k] = __floats2bfloat162_rn(vals[ps][2 * k] * scale * gain[ps][2 * k], vals[ps][2 * k + 1] * scale * gain[ps][2 * k + 1]);
    *reinterpret_cast<uint4*>(p.act_out + (size_t)t * p.C + h) = nb[ps];
  }
  route_partial_logits<MAX_PASSES>(nb, true, r.wg, r.E, p.C, rs);
  __syncthreads();
  for (int e = tid; e < r.E; e += blockDim.x) rs.logit[e] = route_sum_logit(rs, e);
  __syncthreads();
  if (tid < 32) {
    select_grouped_warp<NR_MAX_E>(rs.logit, r.E, r.topk, rule, sel_id, sel_w);
    __syncwarp();
    if (tid == 0) {
      for (int j = 0; j < r.topk; ++j) {
        r.expert_ids[t * r.topk + j] = sel_id[j];
        r.expert_w[t * r.topk + j] = sel_w[j];
      }
      route_publish_and_wait(r, p.status, t, T, rs);
    }
  }
  __syncthreads();
  if (!rs.barrier_ok) return;   // the counters stay dirty: the host clears them when it handles the status
  route_scatter<MAX_PASSES>(r, nb, true, p.C, t, T, rs);
}

template <typename T>
static int add_norm_go(const AddNormParams& p, int B, cudaStream_t s) {
  const bool v4 = p.C % 4 == 0;
  const int units = v4 ? p.C / 4 : p.C;
  // few rows: one access per thread, so that a row's latency is that of one; many rows: smaller CTAs
  int th = 128;
  while (th < (B <= 512 ? 1024 : 256) && th < units) th *= 2;
  if (units > 2 * th && th > 512) th = 512;
  if (v4 && units <= th * 8) {
    const int passes = (units + th - 1) / th;
    auto go = [&](auto fn) -> int { return (int)launch_pdl(fn, dim3(B), dim3(th), 0, s, p); };
    if (passes <= 1) return go(add_norm_kernel<T, 4, 1>);
    if (passes <= 2) return go(add_norm_kernel<T, 4, 2>);
    if (passes <= 4) return go(add_norm_kernel<T, 4, 4>);
    return go(add_norm_kernel<T, 4, 8>);
  }
  const size_t sm = (size_t)p.C * 4;
  if (sm > 200 * 1024) return -1;
  auto fn = v4 ? add_norm_kernel<T, 4, 0> : add_norm_kernel<T, 1, 0>;
  if (sm > 46 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl(fn, dim3(B), dim3(th), sm, s, p);
}

template <typename T>
static int depth_norm_go(const DepthNormParams& p, cudaStream_t s) {
  // few rows: one per CTA; many: runs of rows, of which only the first needs the row before it once more
  int rows = p.shift ? (p.T + 591) / 592 : 1;
  if (rows > 16) rows = 16;
  const dim3 grid((p.T + rows - 1) / rows);
  if (p.C / p.groups % DN_SEG == 0 && p.C <= DN_MAX_SEGS * DN_SEG) {
    // few rows: one access per thread, so that a row's latency is that of one; many rows: smaller CTAs
    int th = 128;
    while (th < (p.T <= 512 || p.C > 4096 ? 512 : 256) && th * 4 < p.C) th *= 2;
    const int passes = (p.C + th * 4 - 1) / (th * 4);
    auto go = [&](auto with, auto without) -> int { return (int)launch_pdl(p.shift ? with : without, grid, dim3(th), 0, s, p, rows); };
    if (passes <= 1) return go(depth_norm_kernel<T, 1, true>, depth_norm_kernel<T, 1, false>);
    if (passes <= 2) return go(depth_norm_kernel<T, 2, true>, depth_norm_kernel<T, 2, false>);
    return go(depth_norm_kernel<T, 4, true>, depth_norm_kernel<T, 4, false>);
  }
  const size_t sm = (size_t)(3 * p.C + p.groups) * 4;
  if (sm > 200 * 1024) return -1;
  if (sm > 46 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(depth_norm_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl(depth_norm_any_kernel<T>, grid, dim3(p.C >= 512 ? 512 : 256), sm, s, p, rows);
}

}  // namespace skein

extern "C" int skein_depth_norm(const SkeinDepthNormParams* p, int fp32, void* stream) {
  using namespace skein;
  if (p->T == 0) return 0;
  if (p->C < 1 || p->groups < 1 || p->C % p->groups != 0 || p->n_terms < 1 || (p->n_terms > 1 && !p->weights)) return -1;
  if (p->shift && (!p->state || !p->positions || !p->slots || (p->seq_of_token && (!p->q_start || !p->q_len)))) return -1;
  return fp32 ? depth_norm_go<float>(*p, (cudaStream_t)stream) : depth_norm_go<__nv_bfloat16>(*p, (cudaStream_t)stream);
}

extern "C" int skein_add_norm(const float* x, const void* y, const int* row_idx, const float* row_w, int topk, const float* step, const float* gain,
                              float* x_out, void* act_out, int B, int C, float eps, int fp32, void* stream) {
  using namespace skein;
  if (B == 0) return 0;
  if (C < 1 || (y != nullptr && (topk < 1 || !row_idx || !row_w)) || (act_out != nullptr && gain == nullptr)) return -1;
  AddNormParams p{x, y, row_idx, row_w, step, gain, x_out, act_out, eps, C, topk};
  return fp32 ? add_norm_go<float>(p, B, (cudaStream_t)stream) : add_norm_go<__nv_bfloat16>(p, B, (cudaStream_t)stream);
}

extern "C" int skein_norm_route(const float* x, const float* gain, void* act_out, float eps, int B, int C, const void* wg, int E, int topk,
                                const SkeinRouteRule* rule, int* expert_ids, float* expert_w, int* counts, int* offsets, int* row_of,
                                int* src_token, void* xs, int* barrier, int max_resident_ctas, int* status, void* stream) {
  using namespace skein;
  if (B == 0) return 0;
  if (C % 8 != 0 || C > 4 * 512 * 8 || E > NR_MAX_E || topk > NR_MAX_K || B * topk > NR_MAX_PAIRS || !route_rule_ok(*rule, E, topk)) return -1;
  if (B > max_resident_ctas) return -2;
  NormRouteParams p{x, gain, (__nv_bfloat16*)act_out, status, eps, C};
  RouteParams r;
  r.wg = (const __nv_bfloat16*)wg; r.expert_ids = expert_ids; r.expert_w = expert_w; r.counts = counts; r.offsets = offsets;
  r.row_of = row_of; r.src_token = src_token; r.xs = (__nv_bfloat16*)xs; r.barrier = barrier;
  r.E = E; r.topk = topk; r.e_first = 0; r.e_count = E;
  r.barrier_budget_ns = (unsigned long long)grid_barrier_budget_ms() * 1000000ull;
  int threads = 64;
  while (threads < 512 && threads * 8 < C) threads *= 2;
  const int passes = (C + threads * 8 - 1) / (threads * 8);
  cudaStream_t s = (cudaStream_t)stream;
  if (passes <= 1) return (int)launch_pdl(norm_route_kernel<1>, dim3(B), dim3(threads), 0, s, p, r, *rule);
  if (passes <= 2) return (int)launch_pdl(norm_route_kernel<2>, dim3(B), dim3(threads), 0, s, p, r, *rule);
  return (int)launch_pdl(norm_route_kernel<4>, dim3(B), dim3(threads), 0, s, p, r, *rule);
}
