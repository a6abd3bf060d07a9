// New tokens of attention layers with rotary positions:
//
//   conv_heads     queries, keys and values behind the projection pass a short causal convolution per channel, queries and keys
//                  are rotated, and all go to their place (query rows, cache pages).  A thread takes four channels over a run
//                  of tokens with the window in registers; the thread of a sequence's first tokens, which reads the kept
//                  projections, also writes the new ones.
//   normed_heads   the same with biased projections, a norm of all queries (all keys) of a token together before the rotation,
//                  and rotated values: a CTA takes the queries, or keys and values, of a run of tokens; sine and cosine
//                  come from a table made once per step
//   rotate_heads   a range of every head's columns rotated, the rest passed on, in the activation type
// Convolution, angles and rotation are fp32 (angles are reduced in fp64).
#include "rotary.cuh"

namespace smc {

constexpr int CH_TOKENS = 16;            // tokens a thread walks
constexpr int CH_MAX_TAPS = 8;

struct ConvHeadsArgs {
  const float* proj;        // [T, ldp]: H * D query, G * D key, G * V value columns (D, V multiples of 4)
  int ldp, H, G, D, V, rot; // the first `rot` columns of query and key heads are rotated
  const float* conv;        // [taps, C], C = all the columns above
  int taps;
  float* hist;              // row r: hist + r * row_stride, [taps - 1, C] projections before the first new token, oldest first
  long long row_stride;
  int n_rows;
  const double* freq;       // [rot / 2]
  const int* positions;
  void* q;                  // [T, H * D]
  void* kpool;              // [n_pages + 1, G * D]
  void* vpool;              // [n_pages + 1, G * V]
  int n_pages;
  const int* locs;
  // normed_heads only
  const float* bias;        // [C]
  const float* qk_norm;     // [H * D + G * D]
  int dim;                  // columns of a head the norms count (the rest are zero)
  float eps;
  const float2* angles;     // [T, ld_angles] {sine, cosine}: `rot` / 2 pairs from qk_first on, V / 2 from v_first on
  int ld_angles, qk_first, v_first, turn;            // the first `turn` columns of value heads are rotated
  Ragged r;
  int* status;
  int pdl;
};

__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float4 fma4(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}

template <int TAPS, typename AT>
__global__ void __launch_bounds__(128) conv_heads_kernel(const ConvHeadsArgs a) {
  constexpr int HL = TAPS - 1;
  const int nq = a.H * a.D, nk = a.G * a.D, C = nq + nk + a.G * a.V, c = (blockIdx.y * 128 + threadIdx.x) * 4;
  float4 w[TAPS];
  if (c < C)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = load4(a.conv + (size_t)j * C + c);
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  if (c >= C) return;
  const RaggedBlock b = ragged_block(a.r, blockIdx.x);
  const int first = blockIdx.z * CH_TOKENS;
  if (first >= b.n) return;
  if (HL > 0 && (b.row < 0 || b.row >= a.n_rows)) {
    if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  const float* src = a.proj + (size_t)b.off * a.ldp + c;
  const int t0 = b.start + first, t1 = b.start + min(b.n, first + CH_TOKENS);
  float4 win[HL > 0 ? HL : 1];                          // win[j]: projection of token t - HL + j
  if (t0 == 0) {
    float* hp = a.hist + (size_t)b.row * a.row_stride + c;
#pragma unroll
    for (int j = 0; j < HL; ++j) win[j] = load4((const float*)hp + (size_t)j * C);
#pragma unroll
    for (int j = 0; j < HL; ++j) {                      // the last HL of old and new ones
      const int t = b.len - HL + j;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (t >= 0) {
        v = load4(src + (size_t)t * a.ldp);
      } else {
#pragma unroll
        for (int q = 0; q < HL; ++q)
          if (q == HL + t) v = win[q];
      }
      store4(hp + (size_t)j * C, v);
    }
  } else {
#pragma unroll
    for (int j = 0; j < HL; ++j) win[j] = load4(src + (size_t)(t0 - HL + j) * a.ldp);       // t0 >= CH_TOKENS > HL
  }
  const int part = c < nq ? 0 : c < nq + nk ? 1 : 2, at = part == 0 ? c : part == 1 ? c - nq : c - nq - nk, col = at % a.D;
  const bool turn = part < 2 && col < a.rot;
  for (int t = t0; t < t1; ++t) {
    const int tok = b.off + t;
    const float4 u = load4(src + (size_t)t * a.ldp);
    float4 y = mul4(w[HL], u);
#pragma unroll
    for (int j = 0; j < HL; ++j) y = fma4(w[j], win[j], y);
#pragma unroll
    for (int j = 0; j + 1 < HL; ++j) win[j] = win[j + 1];
    if (HL > 0) win[HL > 0 ? HL - 1 : 0] = u;
    if (turn) {
      const int p = a.positions[tok];
      const float2 lo = rotate_pair(make_float2(y.x, y.y), a.freq, col >> 1, p);
      y.x = lo.x; y.y = lo.y;
      if (col + 2 < a.rot) {
        const float2 hi = rotate_pair(make_float2(y.z, y.w), a.freq, (col >> 1) + 1, p);
        y.z = hi.x; y.w = hi.y;
      }
    }
    if (part == 0) {
      store4(reinterpret_cast<AT*>(a.q) + (size_t)tok * nq + at, y);
      continue;
    }
    int page = a.locs[tok];
    if (page < 0 || page > a.n_pages) { atomicOr(a.status, SMC_ERR_BOUNDS); page = 0; }
    if (part == 1) store4(reinterpret_cast<AT*>(a.kpool) + (size_t)page * nk + at, y);
    else store4(reinterpret_cast<AT*>(a.vpool) + (size_t)page * (a.G * a.V) + at, y);
  }
}

__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float2 turn_by(float x, float y, float2 sc) { return make_float2(x * sc.y - y * sc.x, y * sc.y + x * sc.x); }

constexpr int NH_THREADS = 512, NH_TOKENS = 8;       // most tokens of a run
constexpr int NH_SMEM = 224 * 1024;                  // seven tokens of the widest rows

// A run of tokens in two passes: convolved columns to shared memory with a sum of squares per token and warp, then norm, rotation and
// stores.  Short runs, so that many CTAs share an SM: the kernel lives from loads in flight.  NV: groups of four columns per thread.
template <int TAPS, int NV, typename AT>
__global__ void __launch_bounds__(NH_THREADS, NV == 1 && TAPS <= 4 ? 2 : 1) normed_heads_kernel(const ConvHeadsArgs a, int run) {
  constexpr int HL = TAPS - 1;
  extern __shared__ __align__(16) float4 nh_y[];     // [run][NV][blockDim.x], every thread reads what it has written
  __shared__ float red[NH_TOKENS][NH_THREADS / 32], scale[NH_TOKENS];
  const int nq = a.H * a.D, nk = a.G * a.D, nv = a.G * a.V, C = nq + nk + nv, nt = blockDim.x;
  const bool keys = blockIdx.y == 1;                 // keys and values, else queries
  const int base = keys ? nq : 0, n = keys ? nk + nv : nq, normed = keys ? nk : nq;      // columns of this CTA, those under the norm
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, live = min(nt >> 5, (n + 127) / 128);
  if (a.pdl) pdl_launch_dependents();
  if (warp >= live) {                                // whole warps without columns; the others meet at a barrier of their own count
    if (a.pdl) pdl_wait_prior_grid();
    return;
  }
  float4 w[NV][TAPS], bias[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * nt) * 4;
    bias[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < n) {
      bias[i] = load4(a.bias + base + c);
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[i][j] = load4(a.conv + (size_t)j * C + base + c);
    }
  }
  if (a.pdl) pdl_wait_prior_grid();
  const RaggedBlock b = ragged_block(a.r, blockIdx.x);
  const int first = blockIdx.z * run;
  if (first >= b.n) return;
  if (HL > 0 && (b.row < 0 || b.row >= a.n_rows)) {
    if (tid == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  const float* src = a.proj + (size_t)b.off * a.ldp + base;
  const int t0 = b.start + first, m = min(b.n - first, run);
  float4 win[NV][HL > 0 ? HL : 1];                   // win[i][j]: biased projection of token t - HL + j
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * nt) * 4;
    if (c >= n) continue;
    float* hp = a.hist + (size_t)b.row * a.row_stride + base + c;
#pragma unroll
    for (int j = 0; j < HL; ++j) {
      const int t = t0 - HL + j;                     // a run is no shorter than the history: only the sequence's first one reads it
      win[i][j] = t >= 0 ? add4(load4(src + (size_t)t * a.ldp + c), bias[i]) : load4((const float*)hp + (size_t)(HL + t) * C);
    }
    if (t0 == 0) {                                   // the last HL of old and new ones; nobody else reads the old ones
#pragma unroll
      for (int j = 0; j < HL; ++j) {
        const int t = b.len - HL + j;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (t >= 0) {
          v = add4(load4(src + (size_t)t * a.ldp + c), bias[i]);
        } else {
#pragma unroll
          for (int q = 0; q < HL; ++q)
            if (q == HL + t) v = win[i][q];
        }
        store4(hp + (size_t)j * C, v);
      }
    }
  }
#pragma unroll 4
  for (int k = 0; k < m; ++k) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (tid + i * nt) * 4;
      if (c >= n) continue;
      const float4 now = add4(load4(src + (size_t)(t0 + k) * a.ldp + c), bias[i]);
      float4 y = mul4(w[i][HL], now);
#pragma unroll
      for (int j = 0; j < HL; ++j) y = fma4(w[i][j], win[i][j], y);
#pragma unroll
      for (int j = 0; j + 1 < HL; ++j) win[i][j] = win[i][j + 1];
      if (HL > 0) win[i][HL > 0 ? HL - 1 : 0] = now;
      nh_y[(k * NV + i) * nt + tid] = y;
      if (c < normed) ss = fmaf(y.x, y.x, fmaf(y.y, y.y, fmaf(y.z, y.z, fmaf(y.w, y.w, ss))));
    }
    ss = warp_sum(ss);
    if (lane == 0) red[k][warp] = ss;
  }
  asm volatile("bar.sync 1, %0;" ::"r"(live * 32) : "memory");
  const float count = (float)((keys ? a.G : a.H) * a.dim);
  for (int k = warp; k < m; k += live) {
    const float ss = warp_sum(lane < live ? red[k][lane] : 0.f);
    if (lane == 0) scale[k] = 1.0f / sqrtf(ss / count + a.eps);
  }
  int pair[NV];                                      // first of the columns' pairs in the table of angles (-1: not rotated)
  bool two[NV];                                      // and the second as well
  float4 g[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * nt) * 4, value = keys && c >= nk;
    const int col = value ? (c - nk) % a.V : c % a.D, rot = value ? a.turn : a.rot;
    pair[i] = col < rot ? (value ? a.v_first : a.qk_first) + (col >> 1) : -1;
    two[i] = col + 2 < rot;
    g[i] = c < normed ? load4(a.qk_norm + base + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  asm volatile("bar.sync 1, %0;" ::"r"(live * 32) : "memory");
#pragma unroll 4
  for (int k = 0; k < m; ++k) {
    const int tok = b.off + t0 + k;
    const float inv = scale[k];
    const float2* ang = a.angles + (size_t)tok * a.ld_angles;
    int page = keys ? a.locs[tok] : 0;
    if (page < 0 || page > a.n_pages) { atomicOr(a.status, SMC_ERR_BOUNDS); page = 0; }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (tid + i * nt) * 4;
      if (c >= n) continue;
      float4 v = nh_y[(k * NV + i) * nt + tid];
      if (c < normed) v = make_float4(v.x * inv * g[i].x, v.y * inv * g[i].y, v.z * inv * g[i].z, v.w * inv * g[i].w);
      if (pair[i] >= 0) {
        const float2 lo = turn_by(v.x, v.y, ang[pair[i]]);
        v.x = lo.x; v.y = lo.y;
        if (two[i]) {
          const float2 hi = turn_by(v.z, v.w, ang[pair[i] + 1]);
          v.z = hi.x; v.w = hi.y;
        }
      }
      AT* out = !keys ? reinterpret_cast<AT*>(a.q) + (size_t)tok * nq + c
                      : c < nk ? reinterpret_cast<AT*>(a.kpool) + (size_t)page * nk + c : reinterpret_cast<AT*>(a.vpool) + (size_t)page * nv + (c - nk);
      store4(out, v);
    }
  }
}

// x [T, ldx] -> out [T, heads * width]; columns [first, first + rot) of every head turn.  A thread takes one pair.
template <typename AT>
__global__ void __launch_bounds__(128) rotate_heads_kernel(const float* x, int ldx, AT* out, int heads, int width, int first, int rot,
                                                           const double* freq, const int* positions, int pdl) {
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int t = blockIdx.x, p = positions[t], n = heads * width / 2;
  const float* row = x + (size_t)t * ldx;
  AT* o = out + (size_t)t * heads * width;
  for (int i = blockIdx.y * 128 + threadIdx.x; i < n; i += gridDim.y * 128) {
    const int c = 2 * i, col = c % width - first;      // `first` may be odd: a pair of columns need not be a pair of the rotation
    float v[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int r = col + k;
      v[k] = row[c + k];
      if (r < 0 || r >= rot) continue;
      const float2 z = rotate_pair((r & 1) ? make_float2(row[c + k - 1], v[k]) : make_float2(v[k], row[c + k + 1]), freq, r >> 1, p);
      v[k] = (r & 1) ? z.y : z.x;
    }
    if constexpr (sizeof(AT) == 2) *reinterpret_cast<__nv_bfloat162*>(o + c) = __floats2bfloat162_rn(v[0], v[1]);
    else *reinterpret_cast<float2*>(o + c) = make_float2(v[0], v[1]);
  }
}

template <typename AT>
static int conv_heads_launch(const ConvHeadsArgs& a, cudaStream_t st) {
  const int C = (a.H + a.G) * a.D + a.G * a.V;
  const dim3 grid(a.r.n_blk, (C / 4 + 127) / 128, (a.r.B + CH_TOKENS - 1) / CH_TOKENS), block(128);
#define SMC_CH(N) case N: return launch_pdl(conv_heads_kernel<N, AT>, grid, block, 0, st, a.pdl, a);
  switch (a.taps) { SMC_CH(1) SMC_CH(2) SMC_CH(3) SMC_CH(4) SMC_CH(5) SMC_CH(6) SMC_CH(7) SMC_CH(8) }
#undef SMC_CH
  return -92;
}

template <typename AT, int NV>
static int normed_heads_taps(const ConvHeadsArgs& a, int threads, cudaStream_t st) {
  int run = a.r.B < NH_TOKENS ? a.r.B : NH_TOKENS;
  if (run > NH_SMEM / (NV * threads * 16)) run = NH_SMEM / (NV * threads * 16);      // seven at the least: as long as any history
  const int smem = run * NV * threads * 16;
  const dim3 grid(a.r.n_blk, 2, (a.r.B + run - 1) / run), block(threads);
#define SMC_NH(N)                                                                                                              \
  case N:                                                                                                                      \
    CUDA_CHECK_RET(cudaFuncSetAttribute(normed_heads_kernel<N, NV, AT>, cudaFuncAttributeMaxDynamicSharedMemorySize, NH_SMEM)); \
    return launch_pdl(normed_heads_kernel<N, NV, AT>, grid, block, smem, st, a.pdl, a, run);
  switch (a.taps) { SMC_NH(1) SMC_NH(2) SMC_NH(3) SMC_NH(4) SMC_NH(5) SMC_NH(6) SMC_NH(7) SMC_NH(8) }
#undef SMC_NH
  return -92;
}

template <typename AT>
static int normed_heads_launch(const ConvHeadsArgs& a, cudaStream_t st) {
  int most = a.H * a.D;
  if (a.G * (a.D + a.V) > most) most = a.G * (a.D + a.V);
  const int groups = (most / 4 + 31) / 32 * 32;
  if (groups <= NH_THREADS) return normed_heads_taps<AT, 1>(a, groups, st);
  if (groups <= NH_THREADS * 2) return normed_heads_taps<AT, 2>(a, NH_THREADS, st);
  if (groups <= NH_THREADS * 4) return normed_heads_taps<AT, 4>(a, NH_THREADS, st);
  return -95;
}

}  // namespace smc

SMC_API int smc_conv_heads_args_size() { return (int)sizeof(smc::ConvHeadsArgs); }

SMC_API int smc_conv_heads(const smc::ConvHeadsArgs* a, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_blk <= 0) return 0;
  if (a->D % 4 || a->V % 4 || a->ldp % 4 || a->rot % 2 || a->rot > a->D || a->taps < 1 || a->taps > CH_MAX_TAPS) return -92;
  return f32 ? conv_heads_launch<float>(*a, st) : conv_heads_launch<__nv_bfloat16>(*a, st);
}

// The normed form (see the top): up to 8192 query columns, as many key and value columns.
SMC_API int smc_normed_heads(const smc::ConvHeadsArgs* a, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_blk <= 0) return 0;
  if (a->D % 4 || a->V % 4 || a->ldp % 4 || a->rot % 2 || a->rot > a->D || a->turn % 2 || a->turn > a->V || a->taps < 1 ||
      a->taps > CH_MAX_TAPS || a->row_stride % 4 || a->angles == nullptr)
    return -92;
  return f32 ? normed_heads_launch<float>(*a, st) : normed_heads_launch<__nv_bfloat16>(*a, st);
}

// Heads of an even number of columns.
SMC_API int smc_rotate_heads(const float* x, int ldx, void* out, int heads, int width, int first, int rot, const double* freq,
                             const int* positions, int T, int f32, int pdl, cudaStream_t st) {
  using namespace smc;
  if (T <= 0) return 0;
  if (width % 2 || rot % 2 || first < 0 || first + rot > width) return -94;
  const int want = (heads * width / 2 + 127) / 128;
  const dim3 grid(T, T >= 296 ? (want + 3) / 4 : want), block(128);
  if (f32) return launch_pdl(rotate_heads_kernel<float>, grid, block, 0, st, pdl, x, ldx, (float*)out, heads, width, first, rot, freq, positions, pdl);
  return launch_pdl(rotate_heads_kernel<__nv_bfloat16>, grid, block, 0, st, pdl, x, ldx, (__nv_bfloat16*)out, heads, width, first, rot, freq,
                    positions, pdl);
}
