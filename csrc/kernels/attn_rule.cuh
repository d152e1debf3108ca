// What a grouped-query attention over the paged cache computes besides q, k and v: mask, sink, number of maps, and what follows the
// softmax (mirrored in skein_b200/ops/_lib.py). Shared by attn_window.cu, attn_decode_mma.cu and attn_prefill_tc.cu.
#pragma once
#include <math.h>
#include <stdint.h>

extern "C" typedef struct SkeinAttnRule {
  const float* lam;          // [1] weight of the second map (maps == 2)
  const void* gate;          // [rows, gate_ld] activation type: the output is multiplied by its sigmoid, or null
  const float* sinks;        // [heads] one more term exp(sinks[h]) in head h's denominator, or null
  int64_t gate_ld;
  int32_t window;            // position i sees j > i - window (0: no window)
  int32_t chunk;             // position i sees j >= i / chunk * chunk (0: no chunks)
  int32_t sink;              // one more term exp(0) in the denominator
  int32_t maps;              // 2: a head is two maps over the same values, o = N(map 1 - lam map 2) with N the division by the root
                             // mean square over the head; query and key heads hold their maps side by side
  int32_t keep_first;        // with a window: position i also sees j < keep_first
  float softcap;             // scores become softcap * tanh(score / softcap) (0: left as they are)
  float scale, out_scale, eps;
  int32_t pad;
} SkeinAttnRule;

// What the append of a step's q, k and v applies per head besides the rotation (each may be null; mirrored in skein_b200/ops/_lib.py).
extern "C" typedef struct SkeinHeadExtras {
  const float *q_bias, *k_bias, *v_bias;     // [heads * dim], [kv_heads * dim], [kv_heads * vdim], added first
  const float *q_norm, *k_norm;              // [dim] weight of an RMS norm of every head, in front of the rotation
  const float* mix;                          // [1] values become (1 - mix) v + mix v_first ...
  const void* v_first;                       // ... with [T, kv_heads * vdim] in the activation type
  void* v_keep;                              // the same layout: where this layer's values go for later layers to mix with
} SkeinHeadExtras;

namespace skein {

// first key that position pos sees
__host__ __device__ __forceinline__ int attn_first_key(int window, int chunk, int pos) {
  if (chunk > 0) return pos / chunk * chunk;
  return window > 0 && pos - window + 1 > 0 ? pos - window + 1 : 0;
}

// the term that a head's sinks add to the softmax's denominator, as a score in base 2 (-infinity: none)
__device__ __forceinline__ float attn_sink_log2(const float* sinks, int head) { return sinks ? sinks[head] * 1.4426950408889634f : -INFINITY; }
__device__ __forceinline__ float attn_sink_log2(const SkeinAttnRule& r, int head) { return r.sink ? 0.f : attn_sink_log2(r.sinks, head); }

// softmax sums (reference m in base 2, denominator l) -> factor that normalises the weighted values
__device__ __forceinline__ float attn_norm(float m, float l, float sink_log2) {
  if (sink_log2 == -INFINITY) return l > 0.f ? 1.f / l : 0.f;
  const float top = fmaxf(m, sink_log2), e = exp2f(m - top);
  return e / (l * e + exp2f(sink_log2 - top));
}

// softcap * tanh(x / softcap) of a raw product s, in base 2: a = 2 scale / softcap and b = softcap, both times log2(e). 1e-7 of b.
__device__ __forceinline__ float attn_cap(float s, float a, float b) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(s * a));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
  return fmaf(-2.f * b, r, b);
}

}  // namespace skein
