// The memories with a decay per channel of memory_scan.cu (kinds channel and forget) for sequences that bring one token each.
//
// A step reads every element of the matrix once, updates it and writes it back: eight threads per value column, each with every
// eighth group of four key rows, and as many CTAs per head (a thread-block cluster) as a round of columns each asks for, so that
// many loads are in flight.  A thread per key row prepares decay, write and read vectors for the whole CTA while the first
// columns are on their way.  The sums of squares of the head's columns meet through distributed shared memory.
#include "memory_scan.cuh"

namespace smc {

constexpr int MS_THREADS = 256;
constexpr int MS_COLS = MS_THREADS / 8;        // columns of one round
constexpr int MS_MAX_COLS = 512;               // of a CTA
constexpr int MS_MAX_KEYS = 256;

template <int KIND, int NK, typename AT>       // NK: groups of four key rows per thread
__global__ void __launch_bounds__(MS_THREADS) memory_step_kernel(const ScanArgs a, int CC, int CS) {
  constexpr bool CHANNEL = KIND == SCAN_CHANNEL;
  __shared__ __align__(16) float s_w[MS_MAX_KEYS], s_k[MS_MAX_KEYS], s_r[MS_MAX_KEYS];
  __shared__ float s_o[MS_MAX_COLS], s_ssq, s_red[2][MS_THREADS / 32];
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int h = blockIdx.x / CS, rank = blockIdx.x - h * CS, s = blockIdx.y, D = a.D, V = a.V;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, sub = tid & 7, c0 = rank * CC, n = min(CC, V - c0);
  const int row = a.r.seq_row[s], t = a.r.seq_off != nullptr ? a.r.seq_off[s] : s;
  if (row < 0 || row >= a.n_rows) {            // the same in every CTA of the cluster
    if (tid == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  const float* p = a.proj + (size_t)t * a.ldp;
  float* M = a.state + (size_t)row * a.row_stride + (size_t)h * V * D;
  float4 m[NK];
  auto fetch = [&](int x) {                    // column x of this CTA
    const float* q = M + (size_t)(c0 + x) * D;
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      const int c = (sub + 8 * i) * 4;
      m[i] = c < D && x < n ? load4(q + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  const int col = tid >> 3;
  fetch(col);
  float b = 1.0f;
  {                                            // operands of key row tid
    const bool ok = tid < D;
    const int at = h * D + tid;
    float k = 0.f, r = 0.f, w = 0.f;
    if (CHANNEL) {
      const int hk = h / a.rep * D + tid;
      k = ok ? p[a.k_off + hk] : 0.f;
      r = ok ? p[a.r_off + hk] : 0.f;
      if (ok) w = expf(-expf(a.a_log[h]) * softplus_f(a.z[(size_t)t * a.ldz + at] + a.w0[at]));
      b = sigmoid_f(a.beta[(size_t)t * a.ldb + h]);
      const float kk = warp_sum(k * k), rr = warp_sum(r * r);
      if (lane == 0) { s_red[0][warp] = kk; s_red[1][warp] = rr; }
      __syncthreads();
      float k2 = 0.f, r2 = 0.f;
#pragma unroll
      for (int i = 0; i < MS_THREADS / 32; ++i) { k2 += s_red[0][i]; r2 += s_red[1][i]; }
      k /= sqrtf(k2 + a.unit_eps);
      r *= a.r_scale / sqrtf(r2 + a.unit_eps);
    } else if (ok) {
      const float z = p[a.a_off + at] + a.a_bias[at], l = a.lower[at];
      r = p[a.r_off + at];
      r *= sigmoid_f(r);
      w = fmaf(1.0f - l, sigmoid_f(z), l);
      k = (1.0f - l) * sigmoid_f(-z);
    }
    s_w[tid] = w;
    s_k[tid] = k;
    s_r[tid] = r;
  }
  __syncthreads();
  float4 w[NK], k[NK], r[NK];
#pragma unroll
  for (int i = 0; i < NK; ++i) {
    const int c = (sub + 8 * i) * 4;
    w[i] = load4((const float*)s_w + c);
    k[i] = load4((const float*)s_k + c);
    r[i] = load4((const float*)s_r + c);
  }
  float sq = 0.f;
  for (int x0 = 0; x0 < CC; x0 += MS_COLS) {   // whole warps stay together
    const int x = x0 + col;
    float* mp = M + (size_t)(c0 + x) * D;
    const bool real = x < n;
    float v = real ? p[a.v_off + h * V + c0 + x] : 0.f, g = 0.f, d = 0.f;
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      m[i] = make_float4(w[i].x * m[i].x, w[i].y * m[i].y, w[i].z * m[i].z, w[i].w * m[i].w);
      if (CHANNEL) g = fmaf(m[i].x, k[i].x, fmaf(m[i].y, k[i].y, fmaf(m[i].z, k[i].z, fmaf(m[i].w, k[i].w, g))));
    }
    if (CHANNEL) {
#pragma unroll
      for (int o = 1; o < 8; o <<= 1) g += __shfl_xor_sync(0xffffffffu, g, o);
      v = b * (v - g);
    }
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      const int c = (sub + 8 * i) * 4;
      m[i] = make_float4(fmaf(v, k[i].x, m[i].x), fmaf(v, k[i].y, m[i].y), fmaf(v, k[i].z, m[i].z), fmaf(v, k[i].w, m[i].w));
      d = fmaf(m[i].x, r[i].x, fmaf(m[i].y, r[i].y, fmaf(m[i].z, r[i].z, fmaf(m[i].w, r[i].w, d))));
      if (real && c < D) store4(mp + c, m[i]);
    }
    if (x0 + MS_COLS < CC) fetch(x + MS_COLS);
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
    if (real && sub == 0) {
      s_o[x] = d;
      sq = fmaf(d, d, sq);
    }
  }
  sq = warp_sum(sq);
  __syncthreads();
  if (lane == 0) s_red[0][warp] = sq;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < MS_THREADS / 32; ++i) tot += s_red[0][i];
  if (CS > 1) {
    if (tid == 0) s_ssq = tot;
    __syncwarp();
    cluster_sync();
    tot = 0.f;
    for (int q = 0; q < CS; ++q) tot += ld_dsmem_f32(smem_u32(&s_ssq), q);
  }
  const float inv = 1.0f / sqrtf(tot / (float)V + a.eps);
  for (int x = tid; x < n; x += MS_THREADS) {
    const int at = h * V + c0 + x;
    float o = s_o[x] * inv * a.onorm[at];
    if (CHANNEL) o *= sigmoid_f(a.gate[(size_t)t * a.ldg + at]);
    reinterpret_cast<AT*>(a.out)[(size_t)t * a.ldo + at] = from_f32<AT>(o);
  }
  __syncwarp();
  if (CS > 1) cluster_sync();                  // nobody leaves while its sum is read
}

template <int KIND, int NK>
static int memory_step_launch(const ScanArgs& a, int f32, cudaStream_t st) {
  int cs = 1;                                  // a round of columns per CTA where the cluster allows it
  while (cs < 8 && cs * MS_COLS < a.V) cs *= 2;
  const int cc = (a.V + cs - 1) / cs;
  if (cc > MS_MAX_COLS) return -122;
  const dim3 grid(a.H * cs, a.r.n_seq), block(MS_THREADS);
  return f32 ? launch_cluster(memory_step_kernel<KIND, NK, float>, grid, block, 0, st, a.pdl, cs, a, cc, cs)
             : launch_cluster(memory_step_kernel<KIND, NK, __nv_bfloat16>, grid, block, 0, st, a.pdl, cs, a, cc, cs);
}

template <int KIND>
static int memory_step_dispatch(const ScanArgs& a, int f32, cudaStream_t st) {
  const int nk = (a.D + 31) / 32;
  if (nk <= 1) return memory_step_launch<KIND, 1>(a, f32, st);
  if (nk <= 2) return memory_step_launch<KIND, 2>(a, f32, st);
  if (nk <= 4) return memory_step_launch<KIND, 4>(a, f32, st);
  return memory_step_launch<KIND, 8>(a, f32, st);
}

}  // namespace smc

// Whether the step takes heads of D key rows (and V value columns).
SMC_API int smc_memory_step_takes(int D, int V) { return D % 4 == 0 && D <= smc::MS_MAX_KEYS && V <= 8 * smc::MS_MAX_COLS; }

// The kinds channel and forget where every sequence brings one token; arguments as for smc_memory_scan.
SMC_API int smc_memory_step(const smc::ScanArgs* a, int kind, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_seq <= 0) return 0;
  if (!smc_memory_step_takes(a->D, a->V) || a->row_stride % 4 || a->H < 1 || a->V < 1 || a->r.n_seq > 65535) return -123;
  if (kind == SCAN_CHANNEL) return a->rep < 1 || a->H % a->rep ? -123 : memory_step_dispatch<SCAN_CHANNEL>(*a, f32, st);
  return kind == SCAN_FORGET ? memory_step_dispatch<SCAN_FORGET>(*a, f32, st) : -123;
}
