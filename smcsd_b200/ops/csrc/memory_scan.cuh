// Arguments shared by the forms of the recurrent memories.
#pragma once
#include "ragged.cuh"

namespace smc {

enum { SCAN_BONUS = 0, SCAN_DELTA = 1, SCAN_GATED = 2 };

struct ScanArgs {
  const float* proj;        // [T, ldp]: H * D columns of r and k, H * V of v and gate at these offsets, from a_off on the removal
  int ldp, r_off, k_off, v_off, g_off, a_off;        // rates (delta, H * D) or the input and forget gates (gated, 2 H)
  const float* z;           // [T, ldz] decay logits, H * D
  int ldz;
  const float* w0;          // [H * D]
  const float* a_bias;      // delta [H * D], gated [2 H]
  const float* bonus;       // wkv
  const float* onorm;       // [H * V]
  float* state;             // row r: state + r * row_stride, [H, V (and one more if gated), D (key)]
  long long row_stride;
  int n_rows;
  void* out;                // [T, ldo]
  int ldo, H, D, V;
  float eps, unit_eps, log_decay;
  float* top;               // gated: row r: top + r * row_stride, [H] running maxima
  float gate_cap, r_scale;  // gated: r is multiplied by r_scale
  Ragged r;
  int* status;
  int pdl;
};

// Gates of the gated form, log domain.
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float log_sigmoid_f(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

}  // namespace smc
