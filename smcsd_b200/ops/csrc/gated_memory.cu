// The gated memory of memory_scan.cu for sequences that bring one token each.
//
// A step reads every element of the matrix once, updates it and writes it back: eight threads per value column, each with every
// eighth group of four key rows, and as many CTAs per head (a thread-block cluster) as fill the machine, so that many loads are in
// flight.  Every CTA takes the normaliser's read-out itself; the first one stores the new normaliser and maximum after all have
// read the old ones.  The sums of squares of the head's columns meet through distributed shared memory.
#include "memory_scan.cuh"

namespace smc {

constexpr int GS_THREADS = 256;
constexpr int GS_COLS = GS_THREADS / 8;        // columns of one round
constexpr int GS_MAX_COLS = 512;               // of a CTA

template <int NK, typename AT>                 // NK: groups of four key rows per thread
__global__ void __launch_bounds__(GS_THREADS) gated_step_kernel(const ScanArgs a, int CC, int CS) {
  __shared__ float s_o[GS_MAX_COLS], s_nq, s_ssq, s_red[GS_THREADS / 32];
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int h = blockIdx.x / CS, rank = blockIdx.x - h * CS, s = blockIdx.y, D = a.D, V = a.V, H = a.H;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, sub = tid & 7, c0 = rank * CC, n = min(CC, V - c0);
  const int row = a.r.seq_row[s], t = a.r.seq_off != nullptr ? a.r.seq_off[s] : s;
  if (row < 0 || row >= a.n_rows) {            // the same in every CTA of the cluster
    if (tid == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  const float* p = a.proj + (size_t)t * a.ldp;
  float* M = a.state + (size_t)row * a.row_stride + (size_t)h * (V + 1) * D;
  float* top = a.top + (size_t)row * a.row_stride + h;
  float4 w[NK], k[NK], q[NK];
  auto fetch = [&](int x) {                    // column x of this CTA
    const float* m = M + (size_t)(c0 + x) * D;
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      const int c = (sub + 8 * i) * 4;
      w[i] = c < D && x < n ? load4(m + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  const int col = tid >> 3;
  fetch(col);
  float kq = 0.f;
#pragma unroll
  for (int i = 0; i < NK; ++i) {
    const int c = (sub + 8 * i) * 4;
    k[i] = q[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < D) {
      k[i] = load4(p + a.k_off + h * D + c);
      q[i] = load4(p + a.r_off + h * D + c);
    }
    q[i] = make_float4(q[i].x * a.r_scale, q[i].y * a.r_scale, q[i].z * a.r_scale, q[i].w * a.r_scale);
    kq = fmaf(k[i].x, q[i].x, fmaf(k[i].y, q[i].y, fmaf(k[i].z, q[i].z, fmaf(k[i].w, q[i].w, kq))));
  }
  // gates, in every thread
  const float cap = a.gate_cap, before = *top;
  const float li = cap * tanhf((p[a.a_off + h] + a.a_bias[h]) / cap);
  const float lf = log_sigmoid_f(cap * tanhf((p[a.a_off + H + h] + a.a_bias[H + h]) / cap));
  const float m = fmaxf(lf + before, li), keep = expf(lf + before - m), add = expf(li - m);
  float4 nrm[NK];                              // the normaliser, by the first eight threads
  if (tid < 8) {
    float d = 0.f;
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      const int c = (sub + 8 * i) * 4;
      nrm[i] = c < D ? load4((const float*)M + (size_t)V * D + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      nrm[i] = make_float4(fmaf(add, k[i].x, keep * nrm[i].x), fmaf(add, k[i].y, keep * nrm[i].y), fmaf(add, k[i].z, keep * nrm[i].z),
                           fmaf(add, k[i].w, keep * nrm[i].w));
      d = fmaf(nrm[i].x, q[i].x, fmaf(nrm[i].y, q[i].y, fmaf(nrm[i].z, q[i].z, fmaf(nrm[i].w, q[i].w, d))));
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) d += __shfl_xor_sync(0xffu, d, o);
    if (tid == 0) s_nq = d;
  }
  float sq = 0.f;
  for (int x0 = 0; x0 < CC; x0 += GS_COLS) {   // whole warps stay together
    const int x = x0 + col;
    float* mp = M + (size_t)(c0 + x) * D;
    const bool real = x < n;
    const float v = real ? add * p[a.v_off + h * V + c0 + x] : 0.f;
    float d = 0.f;
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      const int c = (sub + 8 * i) * 4;
      w[i] = make_float4(fmaf(v, k[i].x, keep * w[i].x), fmaf(v, k[i].y, keep * w[i].y), fmaf(v, k[i].z, keep * w[i].z),
                         fmaf(v, k[i].w, keep * w[i].w));
      d = fmaf(w[i].x, q[i].x, fmaf(w[i].y, q[i].y, fmaf(w[i].z, q[i].z, fmaf(w[i].w, q[i].w, d))));
      if (real && c < D) store4(mp + c, w[i]);
    }
    if (x0 + GS_COLS < CC) fetch(x + GS_COLS);
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
    if (real && sub == 0) {
      s_o[x] = d;
      sq = fmaf(d, d, sq);
    }
  }
  sq = warp_sum(sq);
  if (lane == 0) s_red[warp] = sq;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < GS_THREADS / 32; ++i) tot += s_red[i];
  if (CS > 1) {
    if (tid == 0) s_ssq = tot;
    __syncwarp();
    cluster_sync();
    tot = 0.f;
    for (int r = 0; r < CS; ++r) tot += ld_dsmem_f32(smem_u32(&s_ssq), r);
  }
  const float unit = 1.0f / (fmaxf(fabsf(s_nq), expf(-m)) + a.unit_eps), inv = unit / sqrtf(tot * unit * unit / (float)V + a.eps);
  for (int x = tid; x < n; x += GS_THREADS) {
    const int at = h * V + c0 + x;
    const float o = s_o[x] * inv * a.onorm[at] * sigmoid_f(p[a.g_off + at]);
    reinterpret_cast<AT*>(a.out)[(size_t)t * a.ldo + at] = from_f32<AT>(o);
  }
  if (rank == 0) {
    if (tid < 8) {
#pragma unroll
      for (int i = 0; i < NK; ++i) {
        const int c = (sub + 8 * i) * 4;
        if (c < D) store4(M + (size_t)V * D + c, nrm[i]);
      }
    }
    if (tid == 0) *top = m;
  }
  __syncwarp();
  if (CS > 1) cluster_sync();                  // nobody leaves while its sum is read
}

template <int NK>
static int gated_step_launch(const ScanArgs& a, int f32, cudaStream_t st) {
  int cs = 1;                                  // a round of columns per CTA where the cluster allows it
  while (cs < 8 && cs * GS_COLS < a.V) cs *= 2;
  const int cc = (a.V + cs - 1) / cs;
  if (cc > GS_MAX_COLS) return -122;
  const dim3 grid(a.H * cs, a.r.n_seq), block(GS_THREADS);
  return f32 ? launch_cluster(gated_step_kernel<NK, float>, grid, block, 0, st, a.pdl, cs, a, cc, cs)
             : launch_cluster(gated_step_kernel<NK, __nv_bfloat16>, grid, block, 0, st, a.pdl, cs, a, cc, cs);
}

}  // namespace smc

// Whether the step takes heads of D key rows (and V value columns).
SMC_API int smc_gated_step_takes(int D, int V) { return D % 4 == 0 && D <= 256 && V <= 8 * smc::GS_MAX_COLS; }

// The gated form where every sequence brings one token; arguments as for smc_memory_scan.
SMC_API int smc_gated_step(const smc::ScanArgs* a, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_seq <= 0) return 0;
  if (!smc_gated_step_takes(a->D, a->V) || (a->ldp | a->k_off | a->r_off) % 4 || a->row_stride % 4 || a->H < 1 || a->r.n_seq > 65535) return -123;
  const int nk = (a->D + 31) / 32;
  if (nk <= 1) return gated_step_launch<1>(*a, f32, st);
  if (nk <= 2) return gated_step_launch<2>(*a, f32, st);
  if (nk <= 4) return gated_step_launch<4>(*a, f32, st);
  return gated_step_launch<8>(*a, f32, st);
}
