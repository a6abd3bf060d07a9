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
  int sink;                 // one more term exp(0) in the softmax sum, without a value
  Ragged r;
  int* status;
  int pdl;
};

// First position the token at position p sees.
__device__ __forceinline__ int chunk_start(int p, int chunk) { return p - p % chunk; }

}  // namespace smc
