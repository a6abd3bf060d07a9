// Residual stream of layers whose mixer and feed-forward run side by side on the same input.
//
//   side_step   one kernel between two layers: x <- x + s1 * mixer output + s2 * feed-forward output (scales per channel; the
//               feed-forward's may be a plain row, a row times a gate per token, the weighted rows of the token's experts, or
//               both), the root mean square of the new row, and the row under two norms: one operand for the next mixer, one
//               for the next feed-forward (and in fp32 for its router).  Its first form starts from the embedding, its last
//               form hands on the row under the final norm alone.
// The stream, the scales, the gate and the norms are fp32.
#include "ragged.cuh"

namespace smc {

constexpr int SIDE_MAXV = 8;             // column groups per thread

struct SideArgs {
  float* x;                       // [T, d]
  int d;
  // embedding start (ids != null) ...
  const int* ids;
  const void* embed;              // [vocab, d]
  int vocab;
  float embed_scale;
  // ... or update with the finished layer's outputs
  const float* y1;                // mixer [T, ldy]
  const float* s1;                // [d]
  const float* y2;                // feed-forward [T, ldy] (optional)
  const float* gate;              // [T] multiplies y2 (optional)
  int ldy;
  const float* ye;                // expert rows [slots, ldye] (optional): sum_k route_w[t, k] ye[route_slot[t, k]]
  int ldye, top;
  const int* route_slot;
  const float* route_w;
  const float* s2;                // [d]
  float eps;
  const float* w1;                // norm of the next mixer (of the head with `final`) -> xa
  const float* w2;                // norm of the next feed-forward (optional) -> xb, n2
  void* xa;                       // [T, ldxa]
  void* xb;
  float* n2;                      // [T, d] (optional)
  int ldxa;
  int final;                      // the stream itself is not written back
  int* status;
  int pdl;
};

template <typename AT, int VEC, int NV>
__global__ void __launch_bounds__(256) side_step_kernel(const SideArgs a) {
  __shared__ float red[32];
  const int d = a.d, t = blockIdx.x;
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  float* x = a.x + (size_t)t * d;
  float v[NV][VEC], ss = 0.f;
  int id = 0;
  if (a.ids != nullptr) {
    id = a.ids[t];
    if (id < 0 || id >= a.vocab) {
      if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
      id = 0;
    }
  }
  const float gate = a.gate != nullptr ? a.gate[t] : 1.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * VEC;
    if (c >= d) continue;
    if (a.ids != nullptr) {
      load_cols<VEC>(v[i], reinterpret_cast<const AT*>(a.embed) + (size_t)id * d + c);
#pragma unroll
      for (int k = 0; k < VEC; ++k) v[i][k] *= a.embed_scale;
    } else {
      float y[VEC], s[VEC];
      load_cols<VEC>(v[i], (const float*)x + c);
      load_cols<VEC>(y, a.y1 + (size_t)t * a.ldy + c);
      load_cols<VEC>(s, a.s1 + c);
#pragma unroll
      for (int k = 0; k < VEC; ++k) v[i][k] = fmaf(s[k], y[k], v[i][k]);
      if (a.s2 != nullptr) {
        float f[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) f[k] = 0.f;
        if (a.y2 != nullptr) {
          load_cols<VEC>(y, a.y2 + (size_t)t * a.ldy + c);
#pragma unroll
          for (int k = 0; k < VEC; ++k) f[k] = gate * y[k];
        }
        if (a.ye != nullptr)
          for (int e = 0; e < a.top; ++e) {
            const float w = a.route_w[(size_t)t * a.top + e];
            load_cols<VEC>(y, a.ye + (size_t)a.route_slot[(size_t)t * a.top + e] * a.ldye + c);
#pragma unroll
            for (int k = 0; k < VEC; ++k) f[k] = fmaf(w, y[k], f[k]);
          }
        load_cols<VEC>(s, a.s2 + c);
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[i][k] = fmaf(s[k], f[k], v[i][k]);
      }
    }
    if (!a.final) store_cols<VEC>(x + c, v[i]);
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss = fmaf(v[i][k], v[i][k], ss);
  }
  const float inv = 1.0f / sqrtf(block_sum_all(ss, red) / (float)d + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * VEC;
    if (c >= d) continue;
    float w[VEC], o[VEC];
    load_cols<VEC>(w, a.w1 + c);
#pragma unroll
    for (int k = 0; k < VEC; ++k) o[k] = v[i][k] * inv * w[k];
    store_cols<VEC>(reinterpret_cast<AT*>(a.xa) + (size_t)t * a.ldxa + c, o);
    if (a.w2 == nullptr) continue;
    load_cols<VEC>(w, a.w2 + c);
#pragma unroll
    for (int k = 0; k < VEC; ++k) o[k] = v[i][k] * inv * w[k];
    store_cols<VEC>(reinterpret_cast<AT*>(a.xb) + (size_t)t * a.ldxa + c, o);
    if (a.n2 != nullptr) store_cols<VEC>(a.n2 + (size_t)t * d + c, o);
  }
}

template <typename AT>
static int side_launch(const SideArgs& a, int T, cudaStream_t st) {
  const bool vec = a.d % 4 == 0 && a.ldy % 4 == 0 && a.ldye % 4 == 0 && a.ldxa % 4 == 0;
  const int groups = vec ? a.d / 4 : a.d;
  const int threads = groups <= 64 ? 64 : groups <= 128 ? 128 : 256;
  if (groups > threads * SIDE_MAXV) return -91;
  const dim3 grid(T), block(threads);
  if (!vec) return launch_pdl(side_step_kernel<AT, 1, SIDE_MAXV>, grid, block, 0, st, a.pdl, a);
  if (groups <= threads) return launch_pdl(side_step_kernel<AT, 4, 1>, grid, block, 0, st, a.pdl, a);
  if (groups <= threads * 2) return launch_pdl(side_step_kernel<AT, 4, 2>, grid, block, 0, st, a.pdl, a);
  return launch_pdl(side_step_kernel<AT, 4, SIDE_MAXV>, grid, block, 0, st, a.pdl, a);
}

}  // namespace smc

SMC_API int smc_side_args_size() { return (int)sizeof(smc::SideArgs); }

// One step of the stream for T tokens (see SideArgs); f32: embeddings and activations are fp32 instead of bf16.
SMC_API int smc_side_step(const smc::SideArgs* a, int T, int f32, cudaStream_t st) {
  using namespace smc;
  if (T <= 0) return 0;
  return f32 ? side_launch<float>(*a, T, st) : side_launch<__nv_bfloat16>(*a, T, st);
}
