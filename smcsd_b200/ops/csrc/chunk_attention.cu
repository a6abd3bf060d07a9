// Attention inside chunks of the sequence, inside a sliding window or over all of it, with grouped heads, unit-rms queries and
// keys, a logarithmic distance bias or soft-capped scores, a sink in the softmax sum, a gate on the output or a rotation of it
// against the token's position.
//
//   heads_new     per new token: queries and keys divided by their root mean square per head, values mixed with the first
//                 layer's; keys and values go to the token's cache page
//   chunk_attn    attention of single tokens (and of everything in 32-bit runs): one CTA per (token, kv head, group of
//                 query heads, key range); a key is read by eight lanes, each of which keeps the softmax state of one query
//                 head, and the 32 key streams of a CTA are merged at the end.  Key ranges of one token are a thread-block
//                 cluster and merge through distributed shared memory.  Prompts in bf16 take the tensor-core form in
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

// Eight consecutive elements as they come from memory, so that the next key's are in flight while this one's are used.
template <typename AT> struct Raw8;
template <> struct Raw8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) { a = load4(p); b = load4(p + 4); }
  __device__ __forceinline__ void clear() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ void get(float (&v)[8]) const {
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
};
template <> struct Raw8<__nv_bfloat16> {
  uint4 a;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { a = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void clear() { a = make_uint4(0, 0, 0, 0); }
  __device__ __forceinline__ void get(float (&v)[8]) const {
    const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      v[2 * i] = __uint_as_float(w[i] << 16);
      v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
  }
};

constexpr int CA_WARPS = 8;

// Sum of s[h] over the eight lanes of a key; lane `sub` receives head sub % RH.
template <int RH> __device__ __forceinline__ float scatter_sum(const float (&s)[RH], int sub) {
  float t;
  if constexpr (RH == 4) {
    const bool b0 = sub & 1, b1 = sub & 2;
    const float x = (b0 ? s[1] : s[0]) + __shfl_xor_sync(0xffffffffu, b0 ? s[0] : s[1], 1);
    const float y = (b0 ? s[3] : s[2]) + __shfl_xor_sync(0xffffffffu, b0 ? s[2] : s[3], 1);
    t = (b1 ? y : x) + __shfl_xor_sync(0xffffffffu, b1 ? x : y, 2);
  } else if constexpr (RH == 2) {
    const bool b0 = sub & 1;
    t = (b0 ? s[1] : s[0]) + __shfl_xor_sync(0xffffffffu, b0 ? s[0] : s[1], 1);
    t += __shfl_xor_sync(0xffffffffu, t, 2);
  } else {
    t = s[0];
    t += __shfl_xor_sync(0xffffffffu, t, 1);
    t += __shfl_xor_sync(0xffffffffu, t, 2);
  }
  return t + __shfl_xor_sync(0xffffffffu, t, 4);
}

// N: groups of 64 columns per head; RH: query heads (of one kv head) per CTA; KS key ranges.
template <typename AT, int N, int RH>
__global__ void __launch_bounds__(CA_WARPS * 32) chunk_attn_kernel(const ChunkAttnArgs a, int KS) {
  __shared__ float s_acc[CA_WARPS][RH][N * 64];
  __shared__ float s_m[CA_WARPS][RH], s_l[CA_WARPS][RH];
  __shared__ float s_o[RH][N * 64], s_ml[2][RH];              // of the CTA
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int unit_id = blockIdx.x / KS, rank = blockIdx.x - unit_id * KS;
  const RaggedBlock b = ragged_block(a.r, unit_id / a.r.B);
  const int i = unit_id % a.r.B, g = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (i >= b.n) return;                                       // the same in every CTA of a cluster, here and below
  const int pos = b.prefix + b.start + i, tok = b.off + b.start + i, rep = a.H / a.G;
  if (b.row < 0 || b.row >= a.bt_rows || b.prefix < 0 || b.prefix + b.len > a.bt_stride) {
    if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  const int sub = lane & 7, unit = warp * 4 + (lane >> 3);
  const int h0 = g * rep + blockIdx.z * RH, nh = min(RH, rep - (int)blockIdx.z * RH), mine = min(sub % RH, nh - 1);
  const int* bt = a.block_table + (size_t)b.row * a.bt_stride;
  const AT* kp = reinterpret_cast<const AT*>(a.kpool) + (size_t)g * a.D;
  const AT* vp = reinterpret_cast<const AT*>(a.vpool) + (size_t)g * a.V;
  const float r1 = a.r1 != nullptr ? a.r1[h0 + mine] : 0.f, r2 = a.r1 != nullptr ? a.r2[h0 + mine] : 0.f;
  const int lo = first_key(a, pos);
  int per = (pos - lo + KS) / KS;
  per = (per + 31) & ~31;
  const int k_begin = lo + rank * per, k_end = min(pos + 1, k_begin + per);
  auto page_of = [&](int k) {
    if (k >= k_end) return -1;
    int page = bt[k];
    if (page < 0 || page > a.n_pages) { atomicOr(a.status, SMC_ERR_BOUNDS); page = 0; }
    return page;
  };
  Raw8<AT> kr[N], vr[N];
  auto fetch = [&](int page) {
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int c = n * 64 + sub * 8;
      if (page >= 0 && c < a.D) kr[n].load(kp + (size_t)page * a.G * a.D + c); else kr[n].clear();
      if (page >= 0 && c < a.V) vr[n].load(vp + (size_t)page * a.G * a.V + c); else vr[n].clear();
    }
  };
  int next = page_of(k_begin + unit);
  fetch(next);
  next = page_of(k_begin + unit + CA_WARPS * 4);
  float q[RH][N][8], acc[RH][N][8], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int h = 0; h < RH; ++h)
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int c = n * 64 + sub * 8;
      Raw8<AT> x;
      if (h < nh && c < a.D) x.load(reinterpret_cast<const AT*>(a.q) + ((size_t)tok * a.H + h0 + h) * a.D + c); else x.clear();
      x.get(q[h][n]);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[h][n][e] = 0.f;
    }
  for (int k0 = k_begin; k0 < k_end; k0 += CA_WARPS * 4) {    // the lanes of a warp stay together
    const int k = k0 + unit;
    float s[RH], vv[N][8];
#pragma unroll
    for (int h = 0; h < RH; ++h) s[h] = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      float kv[8];
      kr[n].get(kv);
      vr[n].get(vv[n]);
#pragma unroll
      for (int h = 0; h < RH; ++h)
#pragma unroll
        for (int e = 0; e < 8; ++e) s[h] = fmaf(q[h][n][e], kv[e], s[h]);
    }
    fetch(next);
    next = page_of(k + 2 * CA_WARPS * 4);
    float sc = scatter_sum<RH>(s, sub) * a.scale;
    if (a.softcap > 0.f) sc = a.softcap * tanhf(sc / a.softcap);
    if (a.r1 != nullptr) sc -= r1 * logf(1.0f + r2 * (float)max(pos - k, 0));
    if (k >= k_end) sc = -INFINITY;
    const float m2 = fmaxf(m, sc), base = m2 == -INFINITY ? 0.f : m2, p = expf(sc - base);
    if (__any_sync(0xffffffffu, m2 > m)) {
      const float f = expf(m - base);
      l *= f;
#pragma unroll
      for (int h = 0; h < RH; ++h) {
        const float fh = __shfl_sync(0xffffffffu, f, (lane & 24) | h);
#pragma unroll
        for (int n = 0; n < N; ++n)
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[h][n][e] *= fh;
      }
      m = m2;
    }
    l += p;
#pragma unroll
    for (int h = 0; h < RH; ++h) {
      const float ph = __shfl_sync(0xffffffffu, p, (lane & 24) | h);
#pragma unroll
      for (int n = 0; n < N; ++n)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[h][n][e] = fmaf(ph, vv[n][e], acc[h][n][e]);
    }
  }
  // four key streams of a warp, then the warps, then the key ranges
  float mw = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 8));
  mw = fmaxf(mw, __shfl_xor_sync(0xffffffffu, mw, 16));
  const float f = mw == -INFINITY ? 0.f : expf(m - mw);
  l *= f;
  l += __shfl_xor_sync(0xffffffffu, l, 8);
  l += __shfl_xor_sync(0xffffffffu, l, 16);
  if (lane < RH) { s_m[warp][lane] = mw; s_l[warp][lane] = l; }
#pragma unroll
  for (int h = 0; h < RH; ++h) {
    const float fh = __shfl_sync(0xffffffffu, f, (lane & 24) | h);
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float v = acc[h][n][e] * fh;
        v += __shfl_xor_sync(0xffffffffu, v, 8);
        v += __shfl_xor_sync(0xffffffffu, v, 16);
        if (lane < 8) s_acc[warp][h][n * 64 + sub * 8 + e] = v;
      }
  }
  __syncthreads();
  for (int x = threadIdx.x; x < nh * a.V; x += CA_WARPS * 32) {
    const int h = x / a.V, c = x - h * a.V;
    float mm = -INFINITY, sum = 0.f, o = 0.f;
#pragma unroll
    for (int w = 0; w < CA_WARPS; ++w) mm = fmaxf(mm, s_m[w][h]);
    const float base = mm == -INFINITY ? 0.f : mm;
#pragma unroll
    for (int w = 0; w < CA_WARPS; ++w) {
      const float fw = expf(s_m[w][h] - base);
      sum = fmaf(s_l[w][h], fw, sum);
      o = fmaf(s_acc[w][h][c], fw, o);
    }
    s_o[h][c] = o;
    if (c == 0) { s_ml[0][h] = mm; s_ml[1][h] = sum; }
  }
  __syncwarp();
  if (KS > 1) cluster_sync(); else __syncthreads();
  for (int x = (threadIdx.x + rank * CA_WARPS * 32) * 2; x < nh * a.V; x += CA_WARPS * 32 * KS * 2) {      // pairs of columns
    const int h = x / a.V, c = x - h * a.V;
    const float extra = a.sink_logit != nullptr ? a.sink_logit[h0 + h] : 0.f;
    float mm = a.sink ? extra : -INFINITY, sum;
    float2 o = make_float2(0.f, 0.f);
    if (KS == 1) {
      mm = fmaxf(mm, s_ml[0][h]);
      const float fq = expf(s_ml[0][h] - mm);
      sum = (a.sink ? expf(extra - mm) : 0.f) + s_ml[1][h] * fq;
      o = make_float2(s_o[h][c] * fq, s_o[h][c + 1] * fq);
    } else {
      const uint32_t am = smem_u32(&s_ml[0][h]), al = smem_u32(&s_ml[1][h]), ao = smem_u32(&s_o[h][c]);
      for (int r = 0; r < KS; ++r) mm = fmaxf(mm, ld_dsmem_f32(am, r));
      sum = a.sink ? expf(extra - mm) : 0.f;
      for (int r = 0; r < KS; ++r) {
        const float fq = expf(ld_dsmem_f32(am, r) - mm);
        sum = fmaf(ld_dsmem_f32(al, r), fq, sum);
        o.x = fmaf(ld_dsmem_f32(ao, r), fq, o.x);
        o.y = fmaf(ld_dsmem_f32(ao + 4, r), fq, o.y);
      }
    }
    o = turn_back(a, tok, c, make_float2(o.x / sum, o.y / sum));
    const int col = (h0 + h) * a.V + c;
    if (a.gate != nullptr) {
      const float* gate = a.gate + (size_t)tok * a.ldg;
      o.x /= 1.0f + expf(-gate[a.gate_heads ? h0 + h : col]);
      o.y /= 1.0f + expf(-gate[a.gate_heads ? h0 + h : col + 1]);
    }
    AT* out = reinterpret_cast<AT*>(a.out) + (size_t)tok * a.H * a.V + col;
    out[0] = from_f32<AT>(o.x);
    out[1] = from_f32<AT>(o.y);
  }
  __syncwarp();
  if (KS > 1) cluster_sync();                                 // nobody leaves while its shared memory is read
}

// Query heads per CTA.
template <typename AT> __host__ constexpr int chunk_heads(int wide, int rep) {
  return wide <= 128 ? (rep >= 3 ? 4 : rep) : wide <= 256 ? (rep >= 2 ? 2 : 1) : 1;
}

template <typename AT>
static int chunk_attn_dispatch(const ChunkAttnArgs& a, int KS, cudaStream_t st) {
  const int wide = a.D > a.V ? a.D : a.V, rep = a.H / a.G, rh = chunk_heads<AT>(wide, rep);
#define SMC_CA(N, RH)                                                                                                     \
  return launch_cluster(chunk_attn_kernel<AT, N, RH>, dim3((unsigned)(a.r.n_blk * a.r.B * KS), a.G, (rep + RH - 1) / RH), \
                        dim3(CA_WARPS * 32), 0, st, a.pdl, KS, a, KS)
  if (wide <= 64) {
    if (rh == 1) SMC_CA(1, 1);
    if (rh == 2) SMC_CA(1, 2);
    SMC_CA(1, 4);
  }
  if (wide <= 128) {
    if (rh == 1) SMC_CA(2, 1);
    if (rh == 2) SMC_CA(2, 2);
    SMC_CA(2, 4);
  }
  if (wide <= 256) {
    if (rh == 1) SMC_CA(4, 1);
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

// Key ranges of the step above for `tokens` tokens that see at most about `keys` keys.
SMC_API int smc_chunk_attn_splits(int tokens, int H, int G, int wide, int keys) {
  const int rep = H / G, rh = smc::chunk_heads<float>(wide, rep);
  const long long ctas = (long long)tokens * G * ((rep + rh - 1) / rh);
  const int slots = wide * rh <= 256 ? 296 : 148;             // one CTA per SM where its registers leave room for no second
  int ks = 1;
  while (ks < 8 && ctas * ks * 2 <= slots && keys / (ks * 2) >= 64) ks *= 2;
  return ks;
}

SMC_API int smc_chunk_attn(const smc::ChunkAttnArgs* a, int splits, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_blk <= 0) return 0;
  if (a->D % 8 || a->V % 8 || a->H % a->G || (a->chunk < 1 && a->window < 1) || a->turn % 2 || splits < 1 || splits > 8) return -110;
  return f32 ? chunk_attn_dispatch<float>(*a, splits, st) : chunk_attn_dispatch<__nv_bfloat16>(*a, splits, st);
}
