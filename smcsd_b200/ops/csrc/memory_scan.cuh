// Arguments shared by the forms of the recurrent memories.
#pragma once
#include "ragged.cuh"

namespace smc {

enum { SCAN_BONUS = 0, SCAN_DELTA = 1, SCAN_GATED = 2, SCAN_CHANNEL = 3, SCAN_FORGET = 4 };

struct ScanArgs {
  const float* proj;        // [T, ldp]: H * D columns of r and k, H * V of v and gate at these offsets, from a_off on the removal
  int ldp, r_off, k_off, v_off, g_off, a_off;        // rates (delta, H * D), the input and forget gates (gated, 2 H) or the
                            // forget gates (forget, H * D)
  const float* z;           // [T, ldz] decay logits, H * D
  int ldz;
  const float* w0;          // [H * D]
  const float* a_bias;      // delta and forget [H * D], gated [2 H]
  const float* bonus;       // wkv
  const float* onorm;       // [H * V]
  float* state;             // row r: state + r * row_stride, [H, V (and one more if gated), D (key)]
  long long row_stride;
  int n_rows;
  void* out;                // [T, ldo]
  int ldo, H, D, V;
  float eps, unit_eps, log_decay;
  float* top;               // gated: row r: top + r * row_stride, [H] running maxima
  float gate_cap, r_scale;  // gated, channel: r is multiplied by r_scale
  const float* beta;        // channel: [T, ldb] logits of the write strength, one per head
  int ldb;
  const float* gate;        // channel: [T, ldg] logits of the output gate, H * V
  int ldg;
  const float* a_log;       // channel: [H] logarithms of the decay rates
  int rep;                  // channel: r and k have H / rep heads
  const float* lower;       // forget: [H * D] lower bounds of the forget gates
  Ragged r;
  int* status;
  int pdl;
};

// Gates of the gated form, log domain.
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float log_sigmoid_f(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

}  // namespace smc
