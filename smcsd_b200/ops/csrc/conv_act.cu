// What stands between the projections of a delta rule with a decay per channel and its memory, in one launch:
//
//   conv   a short causal convolution of queries, keys and values per channel, then silu.  A thread walks a run of tokens with the
//          window in registers; the thread of a sequence's first tokens, which reads the kept projections, also writes the new ones.
//   low    the inputs of the two low-rank maps (decay, output gate): few tokens are multiplied out here, a thread per output; for
//          more the inputs are handed on in the activation type, as the operands of two GEMMs.
// Convolution, its activation and all sums are fp32; the maps' inputs are rounded to the activation type in both forms.
#include "memory_scan.cuh"

namespace smc {

constexpr int CA_TOKENS = 16, CA_THREADS = 128, CA_MAX_TAPS = 8;

struct ConvActArgs {
  const float* proj;        // [T, ldp], the first C columns pass the convolution
  int ldp, C;
  const float* conv;        // [taps, C]
  int taps;
  float* hist;              // row r: hist + r * row_stride, [taps - 1, C] projections before the first new token, oldest first
  long long row_stride;
  int n_rows;
  float* out;               // [T, ldo]
  int ldo;
  int low_off, k1, k2;      // inputs of the maps: columns [low_off, + k1) and [.. + k1, + k2) of proj
  void* low;                // [T, k1 + k2] in the activation type, or null: multiply out
  const void* w1;           // [n1, k1]
  const void* w2;           // [n2, k2]
  float* z1;                // [T, n1]
  float* z2;                // [T, n2]
  int n1, n2;
  Ragged r;
  int* status;
  int pdl;
};

template <int TAPS, int VEC, typename AT>
__global__ void __launch_bounds__(CA_THREADS) conv_act_kernel(const ConvActArgs a, int conv_ctas) {
  constexpr int HL = TAPS - 1;
  extern __shared__ __align__(16) float ca_smem[];
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const RaggedBlock b = ragged_block(a.r, blockIdx.x);
  const int first = blockIdx.z * CA_TOKENS;
  if (first >= b.n) return;
  const int t0 = b.start + first, t1 = b.start + min(b.n, first + CA_TOKENS);
  if ((int)blockIdx.y >= conv_ctas) {                   // ---- low
    const int x = (blockIdx.y - conv_ctas) * CA_THREADS + threadIdx.x, k = a.k1 + a.k2;
    if (a.low != nullptr) {
      const int c = x * 4;
      if (c >= k) return;
      for (int t = t0; t < t1; ++t)
        store4(reinterpret_cast<AT*>(a.low) + (size_t)(b.off + t) * k + c, load4(a.proj + (size_t)(b.off + t) * a.ldp + a.low_off + c));
      return;
    }
    const bool second = x >= a.n1;
    const int o = second ? x - a.n1 : x, kk = second ? a.k2 : a.k1;
    const bool real = x < a.n1 + a.n2;
    const AT* w = reinterpret_cast<const AT*>(second ? a.w2 : a.w1) + (size_t)(real ? o : 0) * kk;
    const float* in = ca_smem + (second ? a.k1 : 0);
    for (int t = t0; t < t1; ++t) {
      __syncthreads();
      for (int c = threadIdx.x; c < k; c += CA_THREADS) ca_smem[c] = to_f32<AT>(from_f32<AT>(a.proj[(size_t)(b.off + t) * a.ldp + a.low_off + c]));
      __syncthreads();
      if (!real) continue;
      float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
      for (int c = 0; c < kk; c += 4) {
        const float4 p = load4(w + c), q = load4(in + c);
        s[0] = fmaf(p.x, q.x, s[0]);
        s[1] = fmaf(p.y, q.y, s[1]);
        s[2] = fmaf(p.z, q.z, s[2]);
        s[3] = fmaf(p.w, q.w, s[3]);
      }
      (second ? a.z2 + (size_t)(b.off + t) * a.n2 : a.z1 + (size_t)(b.off + t) * a.n1)[o] = (s[0] + s[1]) + (s[2] + s[3]);
    }
    return;
  }
  // ---- conv
  const int c = (blockIdx.y * CA_THREADS + threadIdx.x) * VEC;
  if (c >= a.C) return;
  if (HL > 0 && (b.row < 0 || b.row >= a.n_rows)) {
    if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  float w[TAPS][VEC], win[HL > 0 ? HL : 1][VEC], u[VEC];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) load_cols<VEC>(w[j], a.conv + (size_t)j * a.C + c);
  const float* src = a.proj + (size_t)b.off * a.ldp + c;
  float* hp = a.hist + (size_t)b.row * a.row_stride + c;
#pragma unroll
  for (int j = 0; j < HL; ++j) {
    const int t = t0 - HL + j;
    if (t >= 0) load_cols<VEC>(win[j], src + (size_t)t * a.ldp);
    else load_cols<VEC>(win[j], (const float*)hp + (size_t)(HL + t) * a.C);
  }
  if (t0 == 0) {                                        // the last HL of old and new ones; nobody else reads the old ones
#pragma unroll
    for (int j = 0; j < HL; ++j) {
      const int t = b.len - HL + j;
      float v[VEC];
      if (t >= 0) {
        load_cols<VEC>(v, src + (size_t)t * a.ldp);
      } else {
#pragma unroll
        for (int q = 0; q < HL; ++q)
          if (q == HL + t)
#pragma unroll
            for (int k = 0; k < VEC; ++k) v[k] = win[q][k];
      }
      store_cols<VEC>(hp + (size_t)j * a.C, v);
    }
  }
  load_cols<VEC>(u, src + (size_t)t0 * a.ldp);
  for (int t = t0; t < t1; ++t) {
    float y[VEC], now[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
      now[k] = u[k];
      y[k] = w[HL][k] * now[k];
#pragma unroll
      for (int j = 0; j < HL; ++j) y[k] = fmaf(w[j][k], win[j][k], y[k]);
    }
    if (t + 1 < t1) load_cols<VEC>(u, src + (size_t)(t + 1) * a.ldp);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
#pragma unroll
      for (int j = 0; j + 1 < HL; ++j) win[j][k] = win[j + 1][k];
      if (HL > 0) win[HL > 0 ? HL - 1 : 0][k] = now[k];
      y[k] *= sigmoid_f(y[k]);
    }
    store_cols<VEC>(a.out + (size_t)(b.off + t) * a.ldo + c, y);
  }
}

template <typename AT>
static int conv_act_launch(const ConvActArgs& a, cudaStream_t st) {
  const bool vec = a.C % 4 == 0 && a.ldo % 4 == 0 && a.row_stride % 4 == 0;
  const int conv_ctas = (a.C / (vec ? 4 : 1) + CA_THREADS - 1) / CA_THREADS, k = a.k1 + a.k2;
  const int low_ctas = ((a.low != nullptr ? k / 4 : a.n1 + a.n2) + CA_THREADS - 1) / CA_THREADS;
  const dim3 grid(a.r.n_blk, conv_ctas + low_ctas, (a.r.B + CA_TOKENS - 1) / CA_TOKENS), block(CA_THREADS);
  const int smem = a.low != nullptr ? 0 : k * 4;
#define SMC_CA(N)                                                                                                   \
  case N:                                                                                                           \
    return vec ? launch_pdl(conv_act_kernel<N, 4, AT>, grid, block, smem, st, a.pdl, a, conv_ctas)                  \
               : launch_pdl(conv_act_kernel<N, 1, AT>, grid, block, smem, st, a.pdl, a, conv_ctas);
  switch (a.taps) { SMC_CA(1) SMC_CA(2) SMC_CA(3) SMC_CA(4) SMC_CA(5) SMC_CA(6) SMC_CA(7) SMC_CA(8) }
#undef SMC_CA
  return -96;
}

}  // namespace smc

SMC_API int smc_conv_act_args_size() { return (int)sizeof(smc::ConvActArgs); }

SMC_API int smc_conv_act(const smc::ConvActArgs* a, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_blk <= 0) return 0;
  if (a->taps < 1 || a->taps > CA_MAX_TAPS || a->ldp % 4 || a->low_off % 4 || a->k1 % 8 || a->k2 % 8 || a->k1 + a->k2 > 8192) return -96;
  return f32 ? conv_act_launch<float>(*a, st) : conv_act_launch<__nv_bfloat16>(*a, st);
}
