// Attention inside chunks of the sequence, with grouped heads, unit-rms queries and keys, a logarithmic distance bias, a sink
// in the softmax sum and a gate on the output.
//
//   heads_new     per new token: queries and keys divided by their root mean square per head, values mixed with the first
//                 layer's; keys and values go to the token's cache page
//   chunk_attn    attention of single tokens (and of everything in 32-bit runs): one CTA per (token, kv head, group of
//                 query heads); a key is read by eight lanes, 16 bytes each, that keep their own softmax state, and the 32
//                 states of a CTA are merged at the end.  Prompts in bf16 take the tensor-core form in
//                 chunk_attention_tc.cu.
#include "chunk_attention.cuh"

namespace smc {

struct HeadsNewArgs {
  const float* proj;        // [T, ldp]: H * D query, G * D key, G * V value columns
  int ldp, H, G, D, V, dim; // dim: columns the mean square is taken over (the rest are zero)
  float eps;
  void* q;                  // [T, H * D]
  void* kpool;
  void* vpool;
  int n_pages;
  const int* locs;
  float lam;                // v <- (1 - lam) v + lam v_first
  float* v_first;           // [T, G * V]
  int gives;                // this layer supplies v_first
  int* status;
  int pdl;
};

template <typename AT>
__global__ void __launch_bounds__(128) heads_new_kernel(const HeadsNewArgs a) {
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float* row = a.proj + (size_t)t * a.ldp;
  int page = a.locs[t];
  if (page < 0 || page > a.n_pages) {
    if (threadIdx.x == 0 && blockIdx.y == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    page = 0;
  }
  const int units = (gridDim.y * 4);
  for (int h = blockIdx.y * 4 + warp; h < a.H + a.G; h += units) {
    const float* src = row + (size_t)h * a.D;
    AT* dst = h < a.H ? reinterpret_cast<AT*>(a.q) + ((size_t)t * a.H + h) * a.D
                      : reinterpret_cast<AT*>(a.kpool) + ((size_t)page * a.G + (h - a.H)) * a.D;
    float ss = 0.f;
    for (int c = lane * 4; c < a.D; c += 128) {
      const float4 v = load4(src + c);
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
    for (int c = lane * 4; c < a.D; c += 128) {
      const float4 v = load4(src + c);
      store4(dst + c, make_float4(v.x * inv, v.y * inv, v.z * inv, v.w * inv));
    }
  }
  const int nv = a.G * a.V;
  const float* src = row + (size_t)(a.H + a.G) * a.D;
  AT* dst = reinterpret_cast<AT*>(a.vpool) + (size_t)page * nv;
  float* first = a.v_first == nullptr ? nullptr : a.v_first + (size_t)t * nv;
  for (int c = (blockIdx.y * 128 + threadIdx.x) * 4; c < nv; c += gridDim.y * 512) {
    float4 v = load4(src + c);
    if (first != nullptr) {
      if (a.gives) {
        store4(first + c, v);
      } else {
        const float4 f = load4((const float*)first + c);
        const float l = a.lam, m = 1.0f - a.lam;
        v = make_float4(m * v.x + l * f.x, m * v.y + l * f.y, m * v.z + l * f.z, m * v.w + l * f.w);
      }
    }
    store4(dst + c, v);
  }
}

template <typename AT> __device__ __forceinline__ void load8(float (&v)[8], const AT* p) {
  const float4 a = load4(p), b = load4(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(float (&v)[8], const __nv_bfloat16* p) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 b = *reinterpret_cast<const __nv_bfloat162*>(&w[i]);
    v[2 * i] = __low2float(b);
    v[2 * i + 1] = __high2float(b);
  }
}

constexpr int CA_WARPS = 8;

// N: groups of 64 columns per head; RH: query heads (of one kv head) per CTA.
template <typename AT, int N, int RH>
__global__ void __launch_bounds__(CA_WARPS * 32) chunk_attn_kernel(const ChunkAttnArgs a) {
  __shared__ float s_acc[CA_WARPS][RH][N * 64];
  __shared__ float s_m[CA_WARPS][RH], s_l[CA_WARPS][RH];
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const RaggedBlock b = ragged_block(a.r, blockIdx.x / a.r.B);
  const int i = blockIdx.x % a.r.B, g = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (i >= b.n) return;
  const int pos = b.prefix + b.start + i, tok = b.off + b.start + i, rep = a.H / a.G;
  if (b.row < 0 || b.row >= a.bt_rows || b.prefix < 0 || b.prefix + b.len > a.bt_stride) {
    if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  const int sub = lane & 7, unit = warp * 4 + (lane >> 3);            // eight lanes share a key
  const int h0 = g * rep + blockIdx.z * RH, nh = min(RH, rep - (int)blockIdx.z * RH);
  const int* bt = a.block_table + (size_t)b.row * a.bt_stride;
  const AT* kp = reinterpret_cast<const AT*>(a.kpool) + (size_t)g * a.D;
  const AT* vp = reinterpret_cast<const AT*>(a.vpool) + (size_t)g * a.V;
  float q[RH][N][8], acc[RH][N][8], m[RH], l[RH], r1[RH], r2[RH];
#pragma unroll
  for (int h = 0; h < RH; ++h) {
    m[h] = -INFINITY;
    l[h] = 0.f;
    r1[h] = (h < nh && a.r1 != nullptr) ? a.r1[h0 + h] : 0.f;
    r2[h] = (h < nh && a.r1 != nullptr) ? a.r2[h0 + h] : 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int c = n * 64 + sub * 8;
#pragma unroll
      for (int e = 0; e < 8; ++e) { q[h][n][e] = 0.f; acc[h][n][e] = 0.f; }
      if (h < nh && c < a.D) load8(q[h][n], reinterpret_cast<const AT*>(a.q) + ((size_t)tok * a.H + h0 + h) * a.D + c);
    }
  }
  const int k_first = chunk_start(pos, a.chunk) + unit;
  int next_page = k_first <= pos ? bt[k_first] : 0;
  for (int k0 = k_first - unit; k0 <= pos; k0 += CA_WARPS * 4) {      // the lanes of a warp stay together
    const int k = k0 + unit;
    const bool live = k <= pos;
    int page = next_page;
    next_page = k + CA_WARPS * 4 <= pos ? bt[k + CA_WARPS * 4] : 0;
    if (page < 0 || page > a.n_pages) { atomicOr(a.status, SMC_ERR_BOUNDS); page = 0; }
    float kv[N][8], vv[N][8];
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int c = n * 64 + sub * 8;
#pragma unroll
      for (int e = 0; e < 8; ++e) { kv[n][e] = 0.f; vv[n][e] = 0.f; }
      if (live && c < a.D) load8(kv[n], kp + (size_t)page * a.G * a.D + c);
      if (live && c < a.V) load8(vv[n], vp + (size_t)page * a.G * a.V + c);
    }
    const float dist = (float)(pos - k);
#pragma unroll
    for (int h = 0; h < RH; ++h) {
      float s = 0.f;
#pragma unroll
      for (int n = 0; n < N; ++n)
#pragma unroll
        for (int e = 0; e < 8; ++e) s = fmaf(q[h][n][e], kv[n][e], s);
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s += __shfl_xor_sync(0xffffffffu, s, 2);
      s += __shfl_xor_sync(0xffffffffu, s, 4);
      if (!live) continue;
      s *= a.scale;
      if (a.r1 != nullptr) s -= r1[h] * logf(1.0f + r2[h] * dist);
      const float m2 = fmaxf(m[h], s), f = expf(m[h] - m2), p = expf(s - m2);
      l[h] = fmaf(l[h], f, p);
      m[h] = m2;
#pragma unroll
      for (int n = 0; n < N; ++n)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[h][n][e] = fmaf(acc[h][n][e], f, p * vv[n][e]);
    }
    __syncwarp();
  }
  // four states of a warp, then the warps
#pragma unroll
  for (int h = 0; h < RH; ++h) {
    float mw = fmaxf(m[h], __shfl_xor_sync(0xffffffffu, m[h], 8));
    mw = fmaxf(mw, __shfl_xor_sync(0xffffffffu, mw, 16));
    const float f = mw == -INFINITY ? 0.f : expf(m[h] - mw);
    float lw = l[h] * f;
    lw += __shfl_xor_sync(0xffffffffu, lw, 8);
    lw += __shfl_xor_sync(0xffffffffu, lw, 16);
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float v = acc[h][n][e] * f;
        v += __shfl_xor_sync(0xffffffffu, v, 8);
        v += __shfl_xor_sync(0xffffffffu, v, 16);
        if (lane < 8) s_acc[warp][h][n * 64 + sub * 8 + e] = v;
      }
    if (lane == 0) { s_m[warp][h] = mw; s_l[warp][h] = lw; }
  }
  __syncthreads();
  for (int x = threadIdx.x; x < nh * a.V; x += CA_WARPS * 32) {
    const int h = x / a.V, c = x - h * a.V;
    float mm = a.sink ? 0.f : -INFINITY;
#pragma unroll
    for (int w = 0; w < CA_WARPS; ++w) mm = fmaxf(mm, s_m[w][h]);
    float sum = a.sink ? expf(-mm) : 0.f, o = 0.f;
#pragma unroll
    for (int w = 0; w < CA_WARPS; ++w) {
      const float f = expf(s_m[w][h] - mm);
      sum = fmaf(s_l[w][h], f, sum);
      o = fmaf(s_acc[w][h][c], f, o);
    }
    o /= sum;
    const int col = (h0 + h) * a.V + c;
    if (a.gate != nullptr) o /= 1.0f + expf(-a.gate[(size_t)tok * a.ldg + col]);
    reinterpret_cast<AT*>(a.out)[(size_t)tok * a.H * a.V + col] = from_f32<AT>(o);
  }
}

template <typename AT>
static int chunk_attn_dispatch(const ChunkAttnArgs& a, cudaStream_t st) {
  const int wide = a.D > a.V ? a.D : a.V, rep = a.H / a.G;
#define SMC_CA(N, RH)                                                                                              \
  return launch_pdl(chunk_attn_kernel<AT, N, RH>, dim3((unsigned)(a.r.n_blk * a.r.B), a.G, (rep + RH - 1) / RH),     \
                    dim3(CA_WARPS * 32), 0, st, a.pdl, a)
  if (wide <= 64) {
    if (rep == 1) SMC_CA(1, 1);
    if (rep == 2) SMC_CA(1, 2);
    SMC_CA(1, 4);
  }
  if (wide <= 128) {
    if (rep == 1) SMC_CA(2, 1);
    if (rep == 2) SMC_CA(2, 2);
    SMC_CA(2, 4);
  }
  if (wide <= 256) {
    if (rep == 1) SMC_CA(4, 1);
    SMC_CA(4, 2);
  }
  if (wide <= 512) SMC_CA(8, 1);
#undef SMC_CA
  return -111;
}

}  // namespace smc

SMC_API int smc_heads_new_args_size() { return (int)sizeof(smc::HeadsNewArgs); }
SMC_API int smc_chunk_attn_args_size() { return (int)sizeof(smc::ChunkAttnArgs); }

SMC_API int smc_heads_new(const smc::HeadsNewArgs* a, int T, int f32, cudaStream_t st) {
  using namespace smc;
  if (T <= 0) return 0;
  if (a->D % 8 || a->V % 8 || a->ldp % 4 || a->dim < 1 || a->dim > a->D) return -110;
  const int want = (a->H + a->G + 3) / 4, split = T >= 296 ? 1 : (want < 16 ? want : 16);      // few tokens: heads over CTAs
  const dim3 grid(T, split), block(128);
  return f32 ? launch_pdl(heads_new_kernel<float>, grid, block, 0, st, a->pdl, *a)
             : launch_pdl(heads_new_kernel<__nv_bfloat16>, grid, block, 0, st, a->pdl, *a);
}

SMC_API int smc_chunk_attn(const smc::ChunkAttnArgs* a, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_blk <= 0) return 0;
  if (a->D % 8 || a->V % 8 || a->H % a->G || a->chunk < 1) return -110;
  return f32 ? chunk_attn_dispatch<float>(*a, st) : chunk_attn_dispatch<__nv_bfloat16>(*a, st);
}
