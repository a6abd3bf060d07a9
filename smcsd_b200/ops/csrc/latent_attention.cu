// Latent attention: every token caches one row of R values that all heads share, as key and (after the value expansion)
// as value.  Queries arrive already multiplied by the key expansion, so a head's score is a dot product of length R with
// the cached row, and the attended rows go through the value expansion afterwards.
//
//   latent_new      per new token: query columns of the projection in the activation type, latent columns divided by their
//                   root mean square (and weighted) into the token's cache page
//   latent_attn     causal attention over the paged rows, one (token, head) per CTA, four warps over the keys: the form
//                   32-bit runs use; the tensor-core form is in latent_attention_tc.cu
#include "latent_attention.cuh"

namespace smc {

template <typename AT>
__global__ void __launch_bounds__(256) latent_new_kernel(const float* proj, int ldp, int nq, int R,
                                                         const float* c_norm, float eps, AT* q,
                                                         int ldq, AT* pool, int ldc, int n_pages,
                                                         const int* cache_locs, int* status, int pdl) {
  __shared__ float red[32];
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int t = blockIdx.x;
  const float* row = proj + (size_t)t * ldp;
  if (q != nullptr) {
    if (((nq | ldp | ldq) & 3) == 0)
      for (int i = threadIdx.x * 4; i < nq; i += blockDim.x * 4) store4(q + (size_t)t * ldq + i, load4(row + i));
    else
      for (int i = threadIdx.x; i < nq; i += blockDim.x) q[(size_t)t * ldq + i] = from_f32<AT>(row[i]);
  }
  const float* c = row + nq;
  float ss = 0.f;
  for (int i = threadIdx.x; i < R; i += blockDim.x) ss = fmaf(c[i], c[i], ss);
  const float inv = 1.0f / sqrtf(block_sum_all(ss, red) / (float)R + eps);
  int page = cache_locs[t];
  if (page < 0 || page > n_pages) {
    if (threadIdx.x == 0) atomicOr(status, SMC_ERR_BOUNDS);
    page = 0;
  }
  for (int i = threadIdx.x; i < R; i += blockDim.x) pool[(size_t)page * ldc + i] = from_f32<AT>(c[i] * inv * c_norm[i]);
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
  for (int k = warp; k < n_keys; k += 4) {
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
  const float mm = fmaxf(fmaxf(s_m[0], s_m[1]), fmaxf(s_m[2], s_m[3]));
  float f[4], lt = 0.f;
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
  switch (a.ldc / 32) { SMC_LA(2) SMC_LA(4) SMC_LA(6) SMC_LA(8) SMC_LA(10) SMC_LA(12) SMC_LA(14) SMC_LA(16) SMC_LA(20) SMC_LA(24) SMC_LA(32) }
#undef SMC_LA
  return -99;
}

}  // namespace smc

SMC_API int smc_latent_args_size() { return (int)sizeof(smc::LatentArgs); }

// proj fp32 [M, ldp]: nq query columns, then R latent columns.  q (optional) [M, ldq]; pool [n_pages + 1, ldc].
SMC_API int smc_latent_new(const float* proj, int ldp, int nq, int R, const float* c_norm, float eps, void* q, int ldq,
                           void* pool, int ldc, int n_pages, const int* cache_locs, int M, int* status, int f32, int pdl,
                           cudaStream_t st) {
  using namespace smc;
  if (M <= 0) return 0;
  if (f32)
    return launch_pdl(latent_new_kernel<float>, dim3(M), dim3(256), 0, st, pdl, proj, ldp, nq, R, c_norm, eps, (float*)q, ldq,
                      (float*)pool, ldc, n_pages, cache_locs, status, pdl);
  return launch_pdl(latent_new_kernel<__nv_bfloat16>, dim3(M), dim3(256), 0, st, pdl, proj, ldp, nq, R, c_norm, eps,
                    (__nv_bfloat16*)q, ldq, (__nv_bfloat16*)pool, ldc, n_pages, cache_locs, status, pdl);
}

SMC_API int smc_latent_attn(const smc::LatentArgs* a, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_blk <= 0) return 0;
  if (a->ldc % 64) return -99;
  return f32 ? latent_attn_dispatch<float>(*a, st) : latent_attn_dispatch<__nv_bfloat16>(*a, st);
}
