// Latent attention: every token caches one row of R values that all heads share, as key and (after the value expansion)
// as value.  Queries arrive already multiplied by the key expansion, so a head's score is a dot product of length R with
// the cached row, and the attended rows go through the value expansion afterwards.
//
//   latent_new      per new token: query columns of the projection in the activation type (or, for queries that go through a
//                   latent of their own, that latent normed), latent columns divided by their root mean square (and weighted)
//                   into the token's cache page, the rotated key behind them
//   latent_attn     causal attention over the paged rows, one (token, head) per CTA, four warps over the keys: the form
//                   32-bit runs use; the tensor-core form is in latent_attention_tc.cu
#include "latent_attention.cuh"
#include "rotary.cuh"

namespace smc {

struct LatentNewArgs {
  const float* proj;        // [T, ldp]: nq query columns, latent columns from c_off on, the rotated key behind them
  int ldp, nq, c_off, R, rot;
  const float* q_norm;      // [nq_real] the query columns are a latent of nq_real values: normed and weighted (null: copied)
  int nq_real;
  const float* c_norm;      // [R]
  float eps;
  const double* freq;       // [rot / 2] angles per position
  const int* positions;
  void* q;                  // [T, ldq] (optional)
  int ldq;
  void* pool;               // [n_pages + 1, ldc]
  int ldc, n_pages;
  const int* locs;
  int* status;
  int pdl;
};

__device__ __forceinline__ int latent_page(const LatentNewArgs& a, int t) {
  const int page = a.locs[t];
  if (page >= 0 && page <= a.n_pages) return page;
  atomicOr(a.status, SMC_ERR_BOUNDS);
  return 0;
}

// Queries copied, no rotated key: a CTA per token.
template <typename AT>
__global__ void __launch_bounds__(256) latent_new_kernel(const LatentNewArgs a) {
  __shared__ float red[32];
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int t = blockIdx.x;
  const float* row = a.proj + (size_t)t * a.ldp;
  AT* q = reinterpret_cast<AT*>(a.q) + (size_t)t * a.ldq;
  if (a.q != nullptr) {
    if (((a.nq | a.ldp | a.ldq) & 3) == 0)
      for (int i = threadIdx.x * 4; i < a.nq; i += blockDim.x * 4) store4(q + i, load4(row + i));
    else
      for (int i = threadIdx.x; i < a.nq; i += blockDim.x) q[i] = from_f32<AT>(row[i]);
  }
  const float* c = row + a.c_off;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.R; i += blockDim.x) ss = fmaf(c[i], c[i], ss);
  const float inv = 1.0f / sqrtf(block_sum_all(ss, red) / (float)a.R + a.eps);
  AT* out = reinterpret_cast<AT*>(a.pool) + (size_t)latent_page(a, t) * a.ldc;
  for (int i = threadIdx.x; i < a.R; i += blockDim.x) out[i] = from_f32<AT>(c[i] * inv * a.c_norm[i]);
}

// Normed query latent and rotated key: a warp per part of a token's row, the values in registers as far as they fit.  VEC: all
// parts start on groups of four columns.
template <typename AT, int VEC>
__global__ void __launch_bounds__(96) latent_rows_kernel(const LatentNewArgs a) {
  constexpr int W = 8;                                    // groups per lane and part
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x;
  const float* row = a.proj + (size_t)t * a.ldp;
  const float* c = row + a.c_off;
  AT* q = reinterpret_cast<AT*>(a.q) + (size_t)t * a.ldq;
  AT* out = reinterpret_cast<AT*>(a.pool) + (size_t)latent_page(a, t) * a.ldc;
  auto unit = [&](AT* dst, const float* src, const float* w, int n) {
    float v[W][VEC], sum = 0.f;
#pragma unroll
    for (int i = 0; i < W; ++i) {
      const int x = (lane + i * 32) * VEC;
      if (x >= n) continue;
      load_cols<VEC>(v[i], src + x);
#pragma unroll
      for (int k = 0; k < VEC; ++k) sum = x + k < n ? fmaf(v[i][k], v[i][k], sum) : sum;
    }
    for (int x = lane + W * 32 * VEC; x < n; x += 32) sum = fmaf(src[x], src[x], sum);
    sum = warp_sum(sum);
    const float inv = 1.0f / sqrtf(sum / (float)n + a.eps);
#pragma unroll
    for (int i = 0; i < W; ++i) {
      const int x = (lane + i * 32) * VEC;
      if (x >= n) continue;
      if (VEC == 1 || x + VEC <= n) {
        float g[VEC];
        load_cols<VEC>(g, w + x);
#pragma unroll
        for (int k = 0; k < VEC; ++k) g[k] *= v[i][k] * inv;
        store_cols<VEC>(dst + x, g);
      } else {
#pragma unroll
        for (int k = 0; k < VEC; ++k)
          if (x + k < n) dst[x + k] = from_f32<AT>(v[i][k] * inv * w[x + k]);
      }
    }
    for (int x = lane + W * 32 * VEC; x < n; x += 32) dst[x] = from_f32<AT>(src[x] * inv * w[x]);
  };
  if (warp == 0) {
    unit(q, row, a.q_norm, a.nq_real);
    for (int x = a.nq_real + lane; x < a.nq; x += 32) q[x] = from_f32<AT>(0.f);
  } else if (warp == 1) {
    unit(out, c, a.c_norm, a.R);
  } else if (a.rot > 0) {
    const int p = a.positions[t];
    for (int i = lane; i < a.rot / 2; i += 32) {
      const float2 v = rotate_pair(make_float2(c[a.R + 2 * i], c[a.R + 2 * i + 1]), a.freq, i, p);
      out[a.R + 2 * i] = from_f32<AT>(v.x);
      out[a.R + 2 * i + 1] = from_f32<AT>(v.y);
    }
  }
}

template <typename AT>
static int latent_new_launch(const LatentNewArgs& a, int T, cudaStream_t st) {
  if (a.q_norm == nullptr) return launch_pdl(latent_new_kernel<AT>, dim3(T), dim3(256), 0, st, a.pdl, a);
  // a group may reach beyond the end of the query latent (zero columns) but not of the cached one, which the rotated key follows
  const bool vec = (a.ldp | a.c_off | a.R | a.ldc | a.ldq | a.nq) % 4 == 0;
  return vec ? launch_pdl(latent_rows_kernel<AT, 4>, dim3(T), dim3(96), 0, st, a.pdl, a)
             : launch_pdl(latent_rows_kernel<AT, 1>, dim3(T), dim3(96), 0, st, a.pdl, a);
}

template <int NR, typename AT>      // NR = ldc / 32 values per lane
__global__ void __launch_bounds__(128) latent_attn_kernel(const LatentArgs a) {
  __shared__ float s_acc[4][NR * 32];
  __shared__ float s_m[4], s_l[4];
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const RaggedBlock b = ragged_block(a.r, blockIdx.x / a.r.B);
  const int i = blockIdx.x % a.r.B, head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (i >= b.n) return;
  if (b.row < 0 || b.row >= a.bt_rows || b.prefix < 0 || b.prefix + b.len > a.bt_stride) {
    if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  const int tok = b.off + b.start + i, n_keys = b.prefix + b.start + i + 1;
  const AT* q = reinterpret_cast<const AT*>(a.q) + ((size_t)tok * a.H + head) * a.ldc;
  const AT* pool = reinterpret_cast<const AT*>(a.pool);
  const int* bt = a.block_table + (size_t)b.row * a.bt_stride;
  float qv[NR], acc[NR], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int j = 0; j < NR; ++j) { qv[j] = to_f32<AT>(q[lane + 32 * j]) * a.scale; acc[j] = 0.f; }
  for (int k = (a.window > 0 ? max(0, n_keys - a.window) : 0) + warp; k < n_keys; k += 4) {
    int page = bt[k];
    if (page < 0 || page > a.n_pages) { atomicOr(a.status, SMC_ERR_BOUNDS); page = 0; }
    const AT* c = pool + (size_t)page * a.ldc;
    float cv[NR], s = 0.f;
#pragma unroll
    for (int j = 0; j < NR; ++j) { cv[j] = to_f32<AT>(c[lane + 32 * j]); s = fmaf(qv[j], cv[j], s); }
    s = warp_sum(s);
    const float m2 = fmaxf(m, s), f = expf(m - m2), p = expf(s - m2);
    l = fmaf(l, f, p);
#pragma unroll
    for (int j = 0; j < NR; ++j) acc[j] = fmaf(acc[j], f, p * cv[j]);
    m = m2;
  }
#pragma unroll
  for (int j = 0; j < NR; ++j) s_acc[warp][lane + 32 * j] = acc[j];
  if (lane == 0) { s_m[warp] = m; s_l[warp] = l; }
  __syncthreads();
  float mm = fmaxf(fmaxf(s_m[0], s_m[1]), fmaxf(s_m[2], s_m[3]));
  if (a.sink != nullptr) mm = fmaxf(mm, a.sink[head]);
  float f[4], lt = a.sink != nullptr ? expf(a.sink[head] - mm) : 0.f;
#pragma unroll
  for (int w = 0; w < 4; ++w) { f[w] = expf(s_m[w] - mm); lt = fmaf(s_l[w], f[w], lt); }
  AT* o = reinterpret_cast<AT*>(a.out) + ((size_t)tok * a.H + head) * a.ldc;
  for (int c = threadIdx.x; c < NR * 32; c += 128)
    o[c] = from_f32<AT>((s_acc[0][c] * f[0] + s_acc[1][c] * f[1] + s_acc[2][c] * f[2] + s_acc[3][c] * f[3]) / lt);
}

template <typename AT>
static int latent_attn_dispatch(const LatentArgs& a, cudaStream_t st) {
  const dim3 grid((unsigned)(a.r.n_blk * a.r.B), (unsigned)a.H), block(128);
#define SMC_LA(NR) case NR: return launch_pdl(latent_attn_kernel<NR, AT>, grid, block, 0, st, a.pdl, a);
  switch (a.ldc / 32) { SMC_LA(2) SMC_LA(4) SMC_LA(6) SMC_LA(8) SMC_LA(10) SMC_LA(12) SMC_LA(14) SMC_LA(16) SMC_LA(18)
                        SMC_LA(20) SMC_LA(22) SMC_LA(24) SMC_LA(26) SMC_LA(28) SMC_LA(30) SMC_LA(32) }
#undef SMC_LA
  return -99;
}

}  // namespace smc

SMC_API int smc_latent_args_size() { return (int)sizeof(smc::LatentArgs); }

SMC_API int smc_latent_new_args_size() { return (int)sizeof(smc::LatentNewArgs); }

SMC_API int smc_latent_new(const smc::LatentNewArgs* a, int T, int f32, cudaStream_t st) {
  using namespace smc;
  if (T <= 0) return 0;
  if (a->rot % 2 || a->R + a->rot > a->ldc || (a->q_norm == nullptr && a->rot != 0) || (a->q_norm != nullptr && a->q == nullptr)) return -98;
  return f32 ? latent_new_launch<float>(*a, T, st) : latent_new_launch<__nv_bfloat16>(*a, T, st);
}

SMC_API int smc_latent_attn(const smc::LatentArgs* a, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_blk <= 0) return 0;
  if (a->ldc % 64) return -99;
  return f32 ? latent_attn_dispatch<float>(*a, st) : latent_attn_dispatch<__nv_bfloat16>(*a, st);
}
