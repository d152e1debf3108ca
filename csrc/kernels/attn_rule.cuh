// What a grouped-query attention over the paged cache computes besides q, k and v: mask, sink, number of maps, and what follows the
// softmax (mirrored in skein_b200/ops/_lib.py). Shared by attn_window.cu, attn_decode_mma.cu and attn_prefill_tc.cu.
#pragma once
#include <math.h>
#include <stdint.h>

extern "C" typedef struct SkeinAttnRule {
  const float* lam;          // [1] weight of the second map (maps == 2)
  const void* gate;          // [rows, gate_ld] activation type: the output is multiplied by its sigmoid, or null
  int64_t gate_ld;
  int32_t window;            // position i sees j > i - window (0: no window)
  int32_t chunk;             // position i sees j >= i / chunk * chunk (0: no chunks)
  int32_t sink;              // one more term exp(0) in the denominator
  int32_t maps;              // 2: a head is two maps over the same values, o = N(map 1 - lam map 2) with N the division by the root
                             // mean square over the head; query and key heads hold their maps side by side
  float scale, out_scale, eps;
  int32_t pad;
} SkeinAttnRule;

namespace skein {

// first key that position pos sees
__host__ __device__ __forceinline__ int attn_first_key(int window, int chunk, int pos) {
  if (chunk > 0) return pos / chunk * chunk;
  return window > 0 && pos - window + 1 > 0 ? pos - window + 1 : 0;
}

}  // namespace skein
