// Parameter blocks of the recurrence kernels (recurrent.cu, recurrent_tc.cu), mirrored in skein_b200/ops/_lib.py (keep the field
// order identical there).
#pragma once
#include <stdint.h>

extern "C" {

typedef struct SkeinRecParams {
  const void* row;           // [rows, ld] projections of the step, activation type
  void* out;                 // [rows, H * V] read-outs, activation type
  float* state;              // [slots, H, D, V]
  void* tail;                // [slots, taps, C] the convolution's last inputs, or null (taps == 1)
  const float* conv_w;       // [taps, C] channels q | k | v; null without a convolution
  const float* conv_b;       // [C] or null
  const float* neg_decay;    // [H] factor of the step in the log decay; lightning: the log decay
  const float* decay;        // [H] lightning: the decay itself, which steps one by one take as it is, or null
  const float* dt_bias;      // [H], [H * D] (channel delta) or null
  const float* skip;         // [H] or null
  const float* step;         // [rows, H * D] inputs of the decays before bias and softplus (channel delta), or null
  const int32_t* positions;  // [rows], -1: padding row
  const int32_t* slots;      // [sequences]
  int32_t* status;
  int64_t ld;
  int32_t kind;              // REC_*
  int32_t H, G, D, V, taps;
  int32_t C;                 // channels of the convolution
  int32_t q_col, k_col, v_col, a_col, b_col;   // first columns in a row: queries, keys, values, decay input, write strength input
  int32_t num_slots;
} SkeinRecParams;

typedef struct SkeinRecChunk {
  const int32_t* seq_of_token;   // [T]
  const int32_t* q_start;        // [S] first row of each sequence's portion
  const int32_t* q_len;          // [S]
  void* qkv;                     // [T, qkv_ld] convolved q | k (2 G D columns) and, from column v_off, v
  float* gates;                  // [T, H, 2] log decay, write coefficient
  float* unit;                   // [T, 2, G] factors of q and k that make unit vectors (delta), or null
  void* chunk_mat;               // scratch of the tensor-core form
  int64_t qkv_ld;
  int32_t v_off;
  int32_t max_q_len;
} SkeinRecChunk;

// A head's output norm and gate (delta rules): o / rms(o) * norm * silu(gate) * scale into out; out null: not applied.
typedef struct SkeinRecGate {
  const float* norm;         // [V]
  void* out;                 // [rows, out_ld]
  const void* gate;          // [rows, gate_ld] H * V columns
  int64_t out_ld, gate_ld;
  int32_t sigmoid;           // the gate's activation is a sigmoid instead of silu
  float eps, scale;
  int32_t pad;
} SkeinRecGate;

}  // extern "C"

namespace skein {
enum : int { REC_DELTA = 0, REC_SSD = 1, REC_LIGHTNING = 2, REC_CHANNEL = 3 };
// the delta rules: what the state holds for k is replaced, q and k are unit vectors
__host__ __device__ constexpr bool rec_corrects(int kind) { return kind == REC_DELTA || kind == REC_CHANNEL; }
using RecParams = SkeinRecParams;
using RecChunk = SkeinRecChunk;
using RecGate = SkeinRecGate;
}  // namespace skein
