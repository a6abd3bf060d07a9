// Residual streams whose norm sits on the sublayers' outputs, and the token shift.
//
//   post_norm_step  one kernel between two sublayers: x <- x + y / rms(y) * w for the finished sublayer's output y, and x in
//                   the activation type for the next one.  Its first form starts from the embedding (token row + sinusoidal
//                   position vector), its last form hands on x / rms(x) * w_final instead.  With single-token sequences the
//                   token shift of the next mixer is folded in: the row before is one row of the state pool.
//   token_shift     the shift on its own (several tokens per sequence): every channel of x is mixed with the row before,
//                   n ways; the thread of a sequence's first tokens, which reads the kept row, also writes the new one.
// The stream, the norms, the angles and the mixes are computed in fp32 (angles are reduced in fp64).
#include "rotary.cuh"

namespace smc {

constexpr int POST_MAXV = 8;             // column groups per thread
constexpr int SHIFT_MAX = 8;             // mixes
constexpr int SHIFT_TOKENS = 16;         // tokens a thread walks

struct PostNormArgs {
  float* x;                       // [T, d]
  int d;
  // embedding start (ids != null) ...
  const int* ids;
  const int* positions;
  const void* embed;              // [vocab, d]
  const double* freq;             // [ceil(d / 2)] angles per position
  int vocab;
  // ... or update with a sublayer's output
  const float* y;                 // [T, ldy]
  int ldy;
  const float* w;                 // [d]
  float eps;
  const float* w_final;           // last step: normalise x, nothing written back
  void* xa;                       // activation rows [T, ldxa] (optional)
  int ldxa;
  // folded token shift (mu != null): token t is the only new token of the sequence with state row rows[t]
  const float* mu;                // [n_mix, d]
  void* mix;                      // [T, n_mix * ldxa]
  float* hist;                    // [n_rows, ldh]
  const int* rows;
  int n_mix, ldh, n_rows;
  int* status;
  int pdl;
};

// AHEAD > 0: AHEAD mixes whose coefficients, and the row before, are read before the sums (two column groups per thread).
template <typename AT, int VEC, int AHEAD>
__global__ void __launch_bounds__(AHEAD ? 512 : 256) post_norm_kernel(const PostNormArgs a) {
  constexpr int POST_MAXV = AHEAD ? 2 : smc::POST_MAXV, NA = AHEAD ? AHEAD : 1, GA = AHEAD ? 2 : 1;
  __shared__ float red[32];
  const int d = a.d, t = blockIdx.x;
  float mus[GA][NA][VEC], before[GA][VEC];
  if constexpr (AHEAD > 0) {
#pragma unroll
    for (int i = 0; i < GA; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * VEC;
      if (c >= d) continue;
#pragma unroll
      for (int s = 0; s < NA; ++s) load_cols<VEC>(mus[i][s], a.mu + (size_t)s * d + c);
    }
  }
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  int row = -1;
  if (a.mu != nullptr) {
    row = a.rows[t];
    if (row < 0 || row >= a.n_rows) {
      if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
      row = -1;
    }
  }
  if constexpr (AHEAD > 0) {
#pragma unroll
    for (int i = 0; i < GA; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * VEC;
      if (c < d && row >= 0) load_cols<VEC>(before[i], (const float*)a.hist + (size_t)row * a.ldh + c);
    }
  }
  float* x = a.x + (size_t)t * d;
  float v[POST_MAXV][VEC];
  if (a.ids != nullptr) {
    int id = a.ids[t], p = a.positions[t];
    if (id < 0 || id >= a.vocab || p < 0) {
      if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
      id = 0;
      p = 0;
    }
    const AT* er = reinterpret_cast<const AT*>(a.embed) + (size_t)id * d;
#pragma unroll
    for (int i = 0; i < POST_MAXV; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * VEC;
      if (c >= d) continue;
      load_cols<VEC>(v[i], er + c);
      if constexpr (VEC == 4) {
        const float2 p0 = position_pair(a.freq, c >> 1, p), p1 = position_pair(a.freq, (c >> 1) + 1, p);
        v[i][0] += p0.x; v[i][1] += p0.y; v[i][2] += p1.x; v[i][3] += p1.y;
      } else {
        const float2 pp = position_pair(a.freq, c >> 1, p);
        v[i][0] += (c & 1) ? pp.y : pp.x;
      }
    }
  } else {
    const float* y = a.y + (size_t)t * a.ldy;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < POST_MAXV; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * VEC;
      if (c >= d) continue;
      load_cols<VEC>(v[i], y + c);
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss = fmaf(v[i][k], v[i][k], ss);
    }
    const float inv = 1.0f / sqrtf(block_sum_all(ss, red) / (float)d + a.eps);
#pragma unroll
    for (int i = 0; i < POST_MAXV; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * VEC;
      if (c >= d) continue;
      float w[VEC], o[VEC];
      load_cols<VEC>(w, a.w + c);
      load_cols<VEC>(o, (const float*)x + c);
#pragma unroll
      for (int k = 0; k < VEC; ++k) v[i][k] = o[k] + v[i][k] * inv * w[k];
    }
  }
  float inv = 0.f;
  if (a.w_final != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < POST_MAXV; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * VEC;
      if (c >= d) continue;
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss = fmaf(v[i][k], v[i][k], ss);
    }
    inv = 1.0f / sqrtf(block_sum_all(ss, red) / (float)d + a.eps);
  }
#pragma unroll
  for (int i = 0; i < POST_MAXV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * VEC;
    if (c >= d) continue;
    if (a.w_final != nullptr) {
      float w[VEC];
      load_cols<VEC>(w, a.w_final + c);
#pragma unroll
      for (int k = 0; k < VEC; ++k) v[i][k] *= inv * w[k];
    } else {
      store_cols<VEC>(x + c, v[i]);
    }
    if (a.xa != nullptr) store_cols<VEC>(reinterpret_cast<AT*>(a.xa) + (size_t)t * a.ldxa + c, v[i]);
    if (row >= 0) {
      float* hp = a.hist + (size_t)row * a.ldh + c;
      AT* m = reinterpret_cast<AT*>(a.mix) + (size_t)t * a.n_mix * a.ldxa + c;
      if constexpr (AHEAD > 0) {
        store_cols<VEC>(hp, v[i]);
#pragma unroll
        for (int s = 0; s < NA; ++s) {
          float o[VEC];
#pragma unroll
          for (int k = 0; k < VEC; ++k) o[k] = fmaf(before[i][k] - v[i][k], mus[i][s][k], v[i][k]);
          store_cols<VEC>(m + (size_t)s * a.ldxa, o);
        }
        continue;
      }
      float back[VEC];
      load_cols<VEC>(back, (const float*)hp);
      store_cols<VEC>(hp, v[i]);
      for (int s = 0; s < a.n_mix; ++s) {
        float mu[VEC], o[VEC];
        load_cols<VEC>(mu, a.mu + (size_t)s * d + c);
#pragma unroll
        for (int k = 0; k < VEC; ++k) o[k] = fmaf(back[k] - v[i][k], mu[k], v[i][k]);
        store_cols<VEC>(m + (size_t)s * a.ldxa, o);
      }
    }
  }
}

template <typename AT, int VEC, int N>
__global__ void __launch_bounds__(128) token_shift_kernel(const float* x, int d, const float* mu, AT* mix, int ldm, float* hist,
                                                          int ldh, int n_rows, const Ragged r, int* status, int pdl) {
  const int c = (blockIdx.y * 128 + threadIdx.x) * VEC;
  float m[N][VEC];
  if (c < d)
#pragma unroll
    for (int s = 0; s < N; ++s) load_cols<VEC>(m[s], mu + (size_t)s * d + c);
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  if (c >= d) return;
  const RaggedBlock b = ragged_block(r, blockIdx.x);
  const int first = blockIdx.z * SHIFT_TOKENS;
  if (first >= b.n) return;
  if (b.row < 0 || b.row >= n_rows) {
    if (threadIdx.x == 0) atomicOr(status, SMC_ERR_BOUNDS);
    return;
  }
  const float* src = x + (size_t)b.off * d + c;
  float back[VEC];
  const int t0 = b.start + first, t1 = b.start + min(b.n, first + SHIFT_TOKENS);
  if (t0 == 0) {
    float* hp = hist + (size_t)b.row * ldh + c;
    float last[VEC];
    load_cols<VEC>(back, (const float*)hp);
    load_cols<VEC>(last, src + (size_t)(b.len - 1) * d);
    store_cols<VEC>(hp, last);
  } else {
    load_cols<VEC>(back, src + (size_t)(t0 - 1) * d);
  }
  for (int t = t0; t < t1; ++t) {
    float v[VEC];
    load_cols<VEC>(v, src + (size_t)t * d);
    AT* o = mix + (size_t)(b.off + t) * N * ldm + c;
#pragma unroll
    for (int s = 0; s < N; ++s) {
      float q[VEC];
#pragma unroll
      for (int k = 0; k < VEC; ++k) q[k] = fmaf(back[k] - v[k], m[s][k], v[k]);
      store_cols<VEC>(o + (size_t)s * ldm, q);
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) back[k] = v[k];
  }
}

template <typename AT>
static int post_norm_launch(const PostNormArgs& a, int T, cudaStream_t st) {
  const bool vec = a.d % 4 == 0 && (a.y == nullptr || a.ldy % 4 == 0) && a.ldxa % 4 == 0 && (a.mu == nullptr || a.ldh % 4 == 0);
  const int groups = vec ? a.d / 4 : a.d;
  const int threads = groups <= 64 ? 64 : groups <= 128 ? 128 : 256;
  if (a.mu != nullptr && a.n_mix == 5 && vec && groups <= 1024)
    return launch_pdl(post_norm_kernel<AT, 4, 5>, dim3(T), dim3(groups <= 512 ? threads : 512), 0, st, a.pdl, a);
  if (groups > threads * POST_MAXV) return -91;
  if (vec) return launch_pdl(post_norm_kernel<AT, 4, 0>, dim3(T), dim3(threads), 0, st, a.pdl, a);
  return launch_pdl(post_norm_kernel<AT, 1, 0>, dim3(T), dim3(threads), 0, st, a.pdl, a);
}

template <typename AT>
static int shift_launch(const float* x, int d, const float* mu, int n, AT* mix, int ldm, float* hist, int ldh, int n_rows,
                        const Ragged& r, int* status, int pdl, cudaStream_t st) {
  const bool vec = d % 4 == 0 && ldm % 4 == 0 && ldh % 4 == 0;
  const int per = 128 * (vec ? 4 : 1);
  const dim3 grid(r.n_blk, (d + per - 1) / per, (r.B + SHIFT_TOKENS - 1) / SHIFT_TOKENS), block(128);
#define SMC_SHIFT(N)                                                                                                            \
  case N:                                                                                                                       \
    return vec ? launch_pdl(token_shift_kernel<AT, 4, N>, grid, block, 0, st, pdl, x, d, mu, mix, ldm, hist, ldh, n_rows, r, status, pdl) \
               : launch_pdl(token_shift_kernel<AT, 1, N>, grid, block, 0, st, pdl, x, d, mu, mix, ldm, hist, ldh, n_rows, r, status, pdl);
  switch (n) { SMC_SHIFT(1) SMC_SHIFT(2) SMC_SHIFT(3) SMC_SHIFT(4) SMC_SHIFT(5) SMC_SHIFT(6) SMC_SHIFT(7) SMC_SHIFT(8) }
#undef SMC_SHIFT
  return -92;
}

}  // namespace smc

SMC_API int smc_post_norm_args_size() { return (int)sizeof(smc::PostNormArgs); }

// One step of the stream for T tokens (see PostNormArgs); f32: embeddings and activations are fp32 instead of bf16.
SMC_API int smc_post_norm_step(const smc::PostNormArgs* a, int T, int f32, cudaStream_t st) {
  using namespace smc;
  if (T <= 0) return 0;
  if (a->mu != nullptr && (a->n_mix < 1 || a->n_mix > SHIFT_MAX)) return -92;
  return f32 ? post_norm_launch<float>(*a, T, st) : post_norm_launch<__nv_bfloat16>(*a, T, st);
}

// mix[t, s, :] = x[t] + (x[t - 1] - x[t]) * mu[s] for the new tokens of every sequence; mix [T, n, ldm], hist [n_rows, ldh]
// holds the row before the first of them and advances.
SMC_API int smc_token_shift(const float* x, int d, const float* mu, int n, void* mix, int ldm, float* hist, int ldh, int n_rows,
                            const smc::Ragged* r, int* status, int f32, int pdl, cudaStream_t st) {
  using namespace smc;
  if (r->n_blk <= 0) return 0;
  if (f32) return shift_launch(x, d, mu, n, (float*)mix, ldm, hist, ldh, n_rows, *r, status, pdl, st);
  return shift_launch(x, d, mu, n, (__nv_bfloat16*)mix, ldm, hist, ldh, n_rows, *r, status, pdl, st);
}
