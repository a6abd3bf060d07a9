// Rotary positions and sinusoids: angles are position times a frequency held in fp64, reduced in fp64.
#pragma once
#include "ragged.cuh"

namespace smc {

// {sine, cosine} of position p at frequency index i.
__device__ __forceinline__ float2 position_pair(const double* freq, int i, int p) {
  double a = (double)p * freq[i];
  a -= 6.283185307179586476925 * rint(a * 0.15915494309189533577);
  float s, c;
  sincosf((float)a, &s, &c);
  return make_float2(s, c);
}

// The neighbouring entries v of a head, pair i, at position p.
__device__ __forceinline__ float2 rotate_pair(float2 v, const double* freq, int i, int p) {
  const float2 sc = position_pair(freq, i, p);
  return make_float2(v.x * sc.y - v.y * sc.x, v.y * sc.y + v.x * sc.x);
}

}  // namespace smc
