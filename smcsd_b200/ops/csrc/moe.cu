// Feed-forward pieces around the GEMMs of layered architectures:
//   poly_norm       a N(z) + b N(z^2) + c N(z^3) + e, N dividing the token's row by its root mean square
//   gated_unit      min(g, limit) sigmoid(slope g) (clamp(u) + shift), or gelu(g) u, on stored gate / up rows (32-bit runs; the
//                   bf16 path has it in the GEMM epilogue)
//   route           router logits (with an optional bias), softmax over all experts, best groups, best experts, renormalised
//                   weights; one more row of the router matrix may give the gate of a shared expert
//   dispatch        slots of the (token, expert) pairs sorted by expert, and the table of token tiles the grouped GEMMs use
//   gather_rows     activation rows in slot order
// Everything the routing decides is fp32.
#include "ragged.cuh"

namespace smc {

// ---------------------------------------------------------------- PolyNorm
template <typename AT>
__global__ void __launch_bounds__(256) poly_norm_kernel(const float* z, int ldz, const float* coef,
                                                        float eps, AT* out, int ldo, int ff, int pdl) {
  __shared__ float red[3][32];
  const float a = coef[0], b = coef[1], c = coef[2], e = coef[3];
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const float* zr = z + (size_t)t * ldz;
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  const bool vec = ((ff | ldz | ldo) & 3) == 0;
  auto add = [&](float v) {
    const float q = v * v, q2 = q * q;
    s1 += q; s2 += q2; s3 = fmaf(q2, q, s3);
  };
  if (vec) {
    for (int i = threadIdx.x * 4; i < ff; i += blockDim.x * 4) {
      const float4 v = load4(zr + i);
      add(v.x); add(v.y); add(v.z); add(v.w);
    }
  } else {
    for (int i = threadIdx.x; i < ff; i += blockDim.x) add(zr[i]);
  }
  s1 = warp_sum(s1); s2 = warp_sum(s2); s3 = warp_sum(s3);
  if (lane == 0) { red[0][warp] = s1; red[1][warp] = s2; red[2][warp] = s3; }
  __syncthreads();
  s1 = warp_sum(lane < nw ? red[0][lane] : 0.f);
  s2 = warp_sum(lane < nw ? red[1][lane] : 0.f);
  s3 = warp_sum(lane < nw ? red[2][lane] : 0.f);
  const float n = (float)ff;
  const float f1 = a / sqrtf(s1 / n + eps), f2 = b / sqrtf(s2 / n + eps), f3 = c / sqrtf(s3 / n + eps);
  auto act = [&](float v) { return fmaf(v, fmaf(v, fmaf(v, f3, f2), f1), e); };
  AT* o = out + (size_t)t * ldo;
  if (vec) {
    for (int i = threadIdx.x * 4; i < ff; i += blockDim.x * 4) {
      const float4 v = load4(zr + i);
      store4(o + i, make_float4(act(v.x), act(v.y), act(v.z), act(v.w)));
    }
  } else {
    for (int i = threadIdx.x; i < ff; i += blockDim.x) o[i] = from_f32<AT>(act(zr[i]));
  }
}

// ---------------------------------------------------------------- gated unit on stored rows (an infinite limit: none)
__global__ void __launch_bounds__(256) gated_unit_kernel(const float* gu, int ldg, float* out, int ldo, int ff, int blk, float limit,
                                                         float slope, float shift, int gelu, int M, int pdl) {
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const long long n = (long long)M * ff;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const int m = (int)(i / ff), c = (int)(i % ff), q = c / blk, r = c - q * blk;
    const float* row = gu + (size_t)m * ldg + (size_t)q * 2 * blk + r;
    const float g = fminf(row[0], limit), u = fminf(fmaxf(row[blk], -limit), limit);
    out[(size_t)m * ldo + c] = gelu ? 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u
                                    : g / (1.0f + expf(-slope * g)) * (u + shift);
  }
}

// ---------------------------------------------------------------- router
// A CTA takes TM tokens; a warp takes four experts at a time, so that a value read from shared memory meets four weight rows
// and their loads overlap (a CTA with one token has more warps, two experts each and more loads in flight).  Then one warp per token runs the softmax and the two selections.
template <typename AT, int TM>
__global__ void __launch_bounds__(TM == 1 ? 1024 : 256) route_kernel(const float* h, int d, const AT* wr, int ldw, int E, int top, int groups,
                                                    int keep, int T, const float* bias, float* gate, int* idx, float* wgt, int pdl) {
  const int EL = E + (gate != nullptr);        // rows of the router matrix
  extern __shared__ float rt_smem[];
  const int d4 = (d + 3) & ~3;
  float* sh = rt_smem;                         // [TM][d4]
  float* sl = sh + (size_t)TM * d4;            // [TM][EL] logits, then scores
  float* sg = sl + TM * EL;                    // [TM][groups] best score of every group
  float* sw = sg + TM * groups;                // [TM][top]
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int t0 = blockIdx.x * TM, nt = min(TM, T - t0), warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const bool vec = (d & 3) == 0 && (ldw & 3) == 0;
  if (vec) {
    for (int i = threadIdx.x * 4; i < TM * d; i += blockDim.x * 4)
      store4(sh + i, i < nt * d ? load4(h + (size_t)t0 * d + i) : make_float4(0.f, 0.f, 0.f, 0.f));
  } else {
    for (int i = threadIdx.x; i < TM * d4; i += blockDim.x) {
      const int m = i / d4, c = i - m * d4;
      sh[i] = m < nt && c < d ? h[(size_t)(t0 + m) * d + c] : 0.f;
    }
  }
  __syncthreads();
  constexpr int EG = TM == 1 ? 2 : 4, AHEAD = TM == 1 ? 8 : 2;
  for (int e0 = warp * EG; e0 < EL; e0 += nw * EG) {
    float acc[EG][TM];
#pragma unroll
    for (int q = 0; q < EG; ++q)
#pragma unroll
      for (int m = 0; m < TM; ++m) acc[q][m] = 0.f;
    if (vec) {
#pragma unroll AHEAD
      for (int c = lane * 4; c < d; c += 128) {
        float4 w[EG];
#pragma unroll
        for (int q = 0; q < EG; ++q) w[q] = load4(wr + (size_t)min(e0 + q, EL - 1) * ldw + c);
#pragma unroll
        for (int m = 0; m < TM; ++m) {
          const float4 v = load4(sh + (size_t)m * d + c);
#pragma unroll
          for (int q = 0; q < EG; ++q)
            acc[q][m] = fmaf(w[q].x, v.x, fmaf(w[q].y, v.y, fmaf(w[q].z, v.z, fmaf(w[q].w, v.w, acc[q][m]))));
        }
      }
    } else {
      for (int c = lane; c < d; c += 32)
#pragma unroll
        for (int q = 0; q < EG; ++q) {
          const float w = to_f32<AT>(wr[(size_t)min(e0 + q, EL - 1) * ldw + c]);
#pragma unroll
          for (int m = 0; m < TM; ++m) acc[q][m] = fmaf(w, sh[(size_t)m * d4 + c], acc[q][m]);
        }
    }
#pragma unroll
    for (int q = 0; q < EG; ++q)
#pragma unroll
      for (int m = 0; m < TM; ++m) {
        const float s = warp_sum(acc[q][m]);
        if (lane == 0 && e0 + q < EL) sl[m * EL + e0 + q] = s + (bias != nullptr && e0 + q < E ? bias[e0 + q] : 0.f);
      }
  }
  __syncthreads();
  const int per = E / groups;
  for (int m = warp; m < nt; m += nw) {
    float* l = sl + m * EL;
    if (gate != nullptr && lane == 0) gate[t0 + m] = 1.0f / (1.0f + expf(-l[E]));
    float* gs = sg + m * groups;
    float mx = -INFINITY;
    for (int e = lane; e < E; e += 32) mx = fmaxf(mx, l[e]);
    mx = warp_max(mx);
    float sum = 0.f;
    for (int e = lane; e < E; e += 32) { const float p = expf(l[e] - mx); l[e] = p; sum += p; }
    sum = warp_sum(sum);
    __syncwarp();
    for (int e = lane; e < E; e += 32) l[e] = l[e] / sum;
    __syncwarp();
    auto argmax = [&](const float* v, int n, float& best, int& at) {      // smallest index among equals
      best = -2.f;
      at = 0x7fffffff;
      for (int i = lane; i < n; i += 32)
        if (v[i] > best) { best = v[i]; at = i; }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float b2 = __shfl_xor_sync(0xffffffffu, best, o);
        const int a2 = __shfl_xor_sync(0xffffffffu, at, o);
        if (b2 > best || (b2 == best && a2 < at)) { best = b2; at = a2; }
      }
    };
    float best;
    int at;
    if (keep < groups) {
      for (int g = lane; g < groups; g += 32) {
        float b = -1.f;
        for (int e = 0; e < per; ++e) b = fmaxf(b, l[g * per + e]);
        gs[g] = b;
      }
      __syncwarp();
      for (int k = 0; k < keep; ++k) {         // a kept group's score moves to [3, 4]: out of the running, marked
        best = -2.f;
        at = 0x7fffffff;
        for (int i = lane; i < groups; i += 32)
          if (gs[i] < 2.f && gs[i] > best) { best = gs[i]; at = i; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
          const float b2 = __shfl_xor_sync(0xffffffffu, best, o);
          const int a2 = __shfl_xor_sync(0xffffffffu, at, o);
          if (b2 > best || (b2 == best && a2 < at)) { best = b2; at = a2; }
        }
        if (lane == 0) gs[at] += 3.f;
        __syncwarp();
      }
      for (int e = lane; e < E; e += 32)
        if (gs[e / per] < 2.f) l[e] = -1.f;
      __syncwarp();
    }
    float tot = 0.f;
    for (int k = 0; k < top; ++k) {
      argmax(l, E, best, at);
      tot += best;
      if (lane == 0) {
        idx[(size_t)(t0 + m) * top + k] = at;
        sw[m * top + k] = best;
        l[at] = -1.f;
      }
      __syncwarp();
    }
    for (int k = lane; k < top; k += 32) wgt[(size_t)(t0 + m) * top + k] = sw[m * top + k] / (tot + 1e-20f);
  }
}

// ---------------------------------------------------------------- dispatch
// One CTA: counts per expert, their prefix sums, a slot for every (token, k) pair, and the tile table
// {expert, first slot, end slot, 0} with at most `rows` slots per entry; unused entries are {0, 0, 0, 0}.
__global__ void __launch_bounds__(1024) dispatch_kernel(const int* idx, int n, int top, int E, int rows,
                                                        int* slot, int* src, int4* tiles,
                                                        int max_tiles, int* status, int pdl) {
  extern __shared__ int dp_smem[];
  int* cnt = dp_smem;                 // [E]
  int* start = cnt + E;               // [E + 1]
  int* tstart = start + E + 1;        // [E + 1]
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int e = idx[i];
    if (e < 0 || e >= E) atomicOr(status, SMC_ERR_BOUNDS);
    else atomicAdd(&cnt[e], 1);
  }
  __syncthreads();
  if (threadIdx.x < 32) {
    int base = 0, tbase = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + threadIdx.x, c = e < E ? cnt[e] : 0, tc = (c + rows - 1) / rows;
      int a = c, b = tc;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int a2 = __shfl_up_sync(0xffffffffu, a, o), b2 = __shfl_up_sync(0xffffffffu, b, o);
        if ((int)threadIdx.x >= o) { a += a2; b += b2; }
      }
      if (e < E) { start[e] = base + a - c; tstart[e] = tbase + b - tc; }
      base += __shfl_sync(0xffffffffu, a, 31);
      tbase += __shfl_sync(0xffffffffu, b, 31);
    }
    if (threadIdx.x == 0) { start[E] = base; tstart[E] = tbase; }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    const int c = cnt[e], s = start[e];
    for (int j = 0, q = tstart[e]; j < c; j += rows, ++q)
      if (q < max_tiles) tiles[q] = make_int4(e, s + j, s + min(j + rows, c), 0);
  }
  for (int q = tstart[E] + threadIdx.x; q < max_tiles; q += blockDim.x) tiles[q] = make_int4(0, 0, 0, 0);
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int e = idx[i];
    int s = 0;
    if (e >= 0 && e < E) {
      s = atomicAdd(&start[e], 1);
      src[s] = i / top;
    }
    slot[i] = s;
  }
}

__global__ void __launch_bounds__(128) gather_rows_kernel(const uint4* x, int ldx16, const int* src,
                                                          uint4* out, int ldo16, int n16, int n_src, int* status,
                                                          int pdl) {
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  int s = src[blockIdx.x];
  if (s < 0 || s >= n_src) {
    if (threadIdx.x == 0) atomicOr(status, SMC_ERR_BOUNDS);
    s = 0;
  }
  for (int i = threadIdx.x; i < n16; i += blockDim.x) out[(size_t)blockIdx.x * ldo16 + i] = x[(size_t)s * ldx16 + i];
}

}  // namespace smc

SMC_API int smc_poly_norm(const float* z, int ldz, const float* coef, float eps, void* out, int ldo, int ff, int M, int f32,
                          int pdl, cudaStream_t st) {
  using namespace smc;
  if (M <= 0) return 0;
  if (f32) return launch_pdl(poly_norm_kernel<float>, dim3(M), dim3(256), 0, st, pdl, z, ldz, coef, eps, (float*)out, ldo, ff, pdl);
  return launch_pdl(poly_norm_kernel<__nv_bfloat16>, dim3(M), dim3(256), 0, st, pdl, z, ldz, coef, eps, (__nv_bfloat16*)out, ldo, ff, pdl);
}

SMC_API int smc_gated_unit_f32(const float* gu, int ldg, float* out, int ldo, int ff, int blk, float limit, float slope,
                               float shift, int gelu, int M, int pdl, cudaStream_t st) {
  using namespace smc;
  if (M <= 0) return 0;
  const long long n = ((long long)M * ff + 255) / 256;
  return launch_pdl(gated_unit_kernel, dim3((unsigned)(n < 2368 ? n : 2368)), dim3(256), 0, st, pdl, gu, ldg, out, ldo, ff, blk,
                    limit, slope, shift, gelu, M, pdl);
}

// h fp32 [T, d] packed; wr [E, ldw]; idx / wgt [T, top].  bias [E] (optional) is added to the logits; gate [T] (optional): wr has
// one more row, the sigmoid of whose logit goes there.
SMC_API int smc_route(const float* h, int d, const void* wr, int ldw, int E, int top, int groups, int keep, int T, const float* bias,
                      float* gate, int* idx, float* wgt, int f32, int pdl, cudaStream_t st) {
  using namespace smc;
  if (T <= 0) return 0;
  if (E < 1 || top < 1 || groups < 1 || E % groups || keep < 1 || keep > groups || top > keep * (E / groups)) return -95;
  auto bytes = [&](int tm) { return (size_t)tm * (((d + 3) & ~3) + E + 1 + groups + top) * sizeof(float); };
  const bool wide = T > 296 && bytes(8) <= 200 * 1024;      // eight tokens per CTA once there are enough of them
  const int TM = wide ? 8 : 1;
  if (bytes(TM) > 200 * 1024) return -96;
  const dim3 grid((T + TM - 1) / TM);
#define SMC_ROUTE(AT, N)                                                                                                    \
  {                                                                                                                         \
    CUDA_CHECK_RET(cudaFuncSetAttribute(route_kernel<AT, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));     \
    return launch_pdl(route_kernel<AT, N>, grid, dim3(N == 1 ? 1024 : 256), bytes(TM), st, pdl, h, d, (const AT*)wr, ldw, E, top, groups,   \
                      keep, T, bias, gate, idx, wgt, pdl);                                                                            \
  }
  if (f32 && wide) SMC_ROUTE(float, 8)
  if (f32) SMC_ROUTE(float, 1)
  if (wide) SMC_ROUTE(__nv_bfloat16, 8)
  SMC_ROUTE(__nv_bfloat16, 1)
#undef SMC_ROUTE
}

// idx [n] expert of every (token, k) pair -> slot [n], src [n] (token of every slot), tiles [max_tiles].
SMC_API int smc_dispatch(const int* idx, int n, int top, int E, int rows, int* slot, int* src, int4* tiles, int max_tiles,
                         int* status, int pdl, cudaStream_t st) {
  using namespace smc;
  if (n <= 0) return 0;
  if (E > 4096 || rows < 1) return -97;
  return launch_pdl(dispatch_kernel, dim3(1), dim3(n > 256 ? 1024 : 256), (size_t)(3 * E + 2) * sizeof(int), st, pdl, idx, n, top, E,
                    rows, slot, src, tiles, max_tiles, status, pdl);
}

// out[i] = x[src[i]]; row pitches and the row length in bytes (multiples of 16).
SMC_API int smc_gather_rows(const void* x, int ldx_bytes, const int* src, void* out, int ldo_bytes, int row_bytes, int n,
                            int n_src, int* status, int pdl, cudaStream_t st) {
  using namespace smc;
  if (n <= 0) return 0;
  if ((ldx_bytes | ldo_bytes | row_bytes) & 15) return -98;
  return launch_pdl(gather_rows_kernel, dim3(n), dim3(128), 0, st, pdl, (const uint4*)x, ldx_bytes / 16, src, (uint4*)out,
                    ldo_bytes / 16, row_bytes / 16, n_src, status, pdl);
}
