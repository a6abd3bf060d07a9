// Arguments shared by the two forms of the chunked attention step.
#pragma once
#include "ragged.cuh"

namespace smc {

struct ChunkAttnArgs {
  const void* q;            // [T, H * D] queries (D, V: head widths padded to multiples of 8, padding columns zero)
  const void* kpool;        // [n_pages + 1, G * D]
  const void* vpool;        // [n_pages + 1, G * V]
  void* out;                // [T, H * V], already multiplied by the gate
  const float* gate;        // [T, ldg]: H * V logits of the output gate (null: no gate)
  int ldg;
  int gate_heads;           // the gate has one logit per head instead
  const int* block_table;
  int bt_stride, bt_rows, n_pages, H, G, D, V;
  int chunk;                // positions of one chunk: a token sees its own chunk only
  float scale;
  const float* r1;          // [H] distance bias r1 ln(1 + r2 distance), taken off the score (null: none)
  const float* r2;
  float softcap;            // score <- softcap tanh(score / softcap) before the bias (0: none)
  int sink;                 // one more term in the softmax sum, without a value: exp(0), or
  const float* sink_logit;  // [H] exp of these
  int window;               // > 0 instead of chunks: a token sees itself and the window - 1 tokens before it
  const float2* angles;     // {sine, cosine} [T, ld_angles]: pair i of an output head turns back by entry angle_first + i (null: not)
  int ld_angles, angle_first, turn;        // the first `turn` columns of a head
  Ragged r;
  int* status;
  int pdl;
};

// First position the token at position p sees.
__device__ __forceinline__ int first_key(const ChunkAttnArgs& a, int p) { return a.window > 0 ? max(0, p - a.window + 1) : p - p % a.chunk; }

// Columns c and c + 1 (a pair) of an output head, turned back by the token's angle.
__device__ __forceinline__ float2 turn_back(const ChunkAttnArgs& a, size_t tok, int c, float2 v) {
  if (a.angles == nullptr || c >= a.turn) return v;
  const float2 sc = a.angles[tok * a.ld_angles + a.angle_first + (c >> 1)];
  return make_float2(v.x * sc.y + v.y * sc.x, v.y * sc.y - v.x * sc.x);
}

}  // namespace smc
