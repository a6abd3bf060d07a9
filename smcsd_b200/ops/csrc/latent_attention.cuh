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
  Ragged r;
  int* status;
  int pdl;
};

}  // namespace smc
