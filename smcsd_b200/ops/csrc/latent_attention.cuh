// Arguments shared by the two forms of the latent attention step.
#pragma once
#include "ragged.cuh"

namespace smc {

struct LatentArgs {
  const void* q;            // [T, H * ldc] queries in latent space (columns beyond R are zero)
  const void* pool;         // [pages + 1, ldc]
  void* out;                // [T, H * ldc]
  const int* block_table;
  int bt_stride, bt_rows, n_pages, H, ldc;
  float scale;
  int window;               // a token sees itself and the window - 1 tokens before it (0: all)
  const float* sink;        // [H] logits in the softmax sum without a value (null: none)
  Ragged r;
  int* status;
  int pdl;
};

}  // namespace smc
