// Recurrent memories: one matrix [key, value] per head, advanced token by token in fp32.
//
//   delta   M <- diag(w) M - (a u)(u^T M) + k v^T, read out with r afterwards; u = k / |k|, a = sigmoid(. + bias),
//           w = exp(-log_decay sigmoid(z + w0)); output gate sigmoid
//   wkv     read out with r before the update, the current k v^T weighted by a bonus; M <- diag(w) M + k v^T,
//           w = exp(-exp(z + w0)); output gate silu
//
// Value columns of a matrix never mix, key rows only in sums.  A CTA therefore keeps some columns of one head's matrix in
// registers - four threads per column, a quarter of the key rows each - and walks its sequence's tokens in tiles: consumer
// warps run the recurrence on the tile in shared memory while four producer warps turn the next tile's projections into
// w, u, a u, ... and finish the outputs of the tile before (division by the head's root mean square, norm weight, gate).
// With few (sequence, head) pairs the columns of a head are spread over a thread-block cluster that exchanges the sums of
// squares through distributed shared memory.  Both sums over key rows are taken over the old matrix, so that a token costs
// one reduction: for delta the read-out is (r w)^T M - (r.a u)(u^T M) + (r.k) v.
// The recurrence is held to fp32 (a bf16 or tf32 chunk-parallel form would round the state), so the floor is the CUDA cores'
// rate; products and sums are issued two at a time (f32x2).
#include "ragged.cuh"

namespace smc {

constexpr int SCAN_PRODUCERS = 4;        // warps

struct ScanArgs {
  const float* proj;        // [T, ldp]: H * D columns each of r, k, v, gate (and removal rate) at these offsets
  int ldp, r_off, k_off, v_off, g_off, a_off;
  const float* z;           // [T, ldz] decay logits, H * D
  int ldz;
  const float* w0;          // [H * D]
  const float* a_bias;      // delta
  const float* bonus;       // wkv
  const float* onorm;       // [H * D]
  float* state;             // row r: state + r * row_stride, [H, D (value), D (key)]
  long long row_stride;
  int n_rows;
  void* out;                // [T, ldo]
  int ldo, H, D;
  float eps, unit_eps, log_decay;
  Ragged r;
  int* status;
  int pdl;
};

typedef unsigned long long f2_t;
__device__ __forceinline__ f2_t pack2(float a, float b) {
  f2_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpack2(f2_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f2_t fma2(f2_t a, f2_t b, f2_t c) {
  f2_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f2_t mul2(f2_t a, f2_t b) {
  f2_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ float sum_of(f2_t a) { const float2 v = unpack2(a); return v.x + v.y; }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }

__host__ __device__ constexpr int scan_tokens(int dkp) { return dkp <= 128 ? 16 : 8; }       // tokens of a tile
__host__ __device__ constexpr int scan_vectors(bool delta) { return delta ? 5 : 3; }

template <bool DELTA, int DKP>
__global__ void __launch_bounds__(640) scan_kernel(const ScanArgs a, int CC, int CS, int f32) {
  constexpr int TB = scan_tokens(DKP), NVEC = scan_vectors(DELTA), NL = (DKP + 31) / 32, NQ = DKP / 16;
  extern __shared__ __align__(16) float scan_smem[];
  const int buf_floats = TB * (NVEC * DKP + CC + 2);
  float* obuf = scan_smem + 2 * buf_floats;                  // [3][TB][CC]
  float* ssq = obuf + 3 * TB * CC;                           // [2][TB]
  const int n_cons = CC * 4, tid = threadIdx.x, lane = tid & 31;
  const bool consumer = tid < n_cons;
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int h = blockIdx.x / CS, rank = blockIdx.x - h * CS, s = blockIdx.y, D = a.D;
  const int row = a.r.seq_row[s];
  const int off = a.r.seq_off != nullptr ? a.r.seq_off[s] : s * a.r.E, len = a.r.seq_len != nullptr ? a.r.seq_len[s] : a.r.E;
  if (row < 0 || row >= a.n_rows) {                          // the same in every CTA of the cluster
    if (tid == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  auto barrier = [&]() {
    __syncwarp();
    if (CS > 1) cluster_sync(); else __syncthreads();
  };
  const int n_tiles = (len + TB - 1) / TB, c0 = rank * CC;

  // ---- producers: one warp per token
  const int pw = (tid - n_cons) >> 5;
  auto stage = [&](int tile) {
    float* buf = scan_smem + (tile & 1) * buf_floats;
    float* val = buf + TB * NVEC * DKP;
    float* scal = val + TB * CC;
    const int n = min(TB, len - tile * TB);
    for (int tb = pw; tb < n; tb += SCAN_PRODUCERS) {
      const size_t t = (size_t)off + tile * TB + tb;
      const float* p = a.proj + t * a.ldp + h * D;
      const float* zr = a.z + t * a.ldz + h * D;
      float kk[NL], rr[NL], zz[NL], aa[NL], ss = 0.f;
#pragma unroll
      for (int i = 0; i < NL; ++i) {
        const int c = lane + 32 * i;
        const bool ok = c < D;
        kk[i] = ok ? p[a.k_off + c] : 0.f;
        rr[i] = ok ? p[a.r_off + c] : 0.f;
        zz[i] = ok ? zr[c] + a.w0[h * D + c] : 0.f;
        aa[i] = ok ? (DELTA ? p[a.a_off + c] + a.a_bias[h * D + c] : a.bonus[h * D + c]) : 0.f;
        ss = fmaf(kk[i], kk[i], ss);
      }
      const float inv = DELTA ? 1.0f / sqrtf(warp_sum(ss) + a.unit_eps) : 0.f;
      float s1 = 0.f, s2 = 0.f;
      float* d = buf + tb * DKP;
#pragma unroll
      for (int i = 0; i < NL; ++i) {
        const int c = lane + 32 * i;
        if (c >= DKP) continue;
        const float w = c >= D ? 0.f : DELTA ? expf(-a.log_decay * sigmoid_f(zz[i])) : expf(-expf(zz[i]));
        d[c] = w;
        d[TB * DKP + c] = kk[i];
        if (DELTA) {
          const float u = kk[i] * inv, au = sigmoid_f(aa[i]) * u;
          d[2 * TB * DKP + c] = rr[i] * w;
          d[3 * TB * DKP + c] = u;
          d[(NVEC - 1) * TB * DKP + c] = au;
          s1 = fmaf(rr[i], au, s1);
          s2 = fmaf(rr[i], kk[i], s2);
        } else {
          d[2 * TB * DKP + c] = rr[i];
          s2 = fmaf(rr[i] * aa[i], kk[i], s2);
        }
      }
      for (int c = lane; c < CC; c += 32) val[tb * CC + c] = c0 + c < D ? p[a.v_off + c0 + c] : 0.f;
      __syncwarp();
      s1 = DELTA ? warp_sum(s1) : 0.f;
      s2 = warp_sum(s2);
      if (lane == 0) { scal[2 * tb] = s1; scal[2 * tb + 1] = s2; }
    }
  };
  auto square = [&](const float* o) {
    float q = 0.f;
    for (int c = lane; c < CC; c += 32) q = fmaf(o[c], o[c], q);
    __syncwarp();
    return warp_sum(q);                                      // columns beyond D are zero
  };
  auto finish = [&](int tile, bool alone) {
    const int n = min(TB, len - tile * TB);
    for (int tb = pw; tb < n; tb += SCAN_PRODUCERS) {
      const size_t t = (size_t)off + tile * TB + tb;
      const float* o = obuf + ((tile % 3) * TB + tb) * CC;
      float tot = 0.f;
      if (alone) {
        tot = square(o);
      } else {
        const uint32_t at = smem_u32(ssq + (tile & 1) * TB + tb);
        for (int q = 0; q < CS; ++q) tot += ld_dsmem_f32(at, q);
      }
      const float inv = 1.0f / sqrtf(tot / (float)D + a.eps);
      for (int c = lane; c < CC && c0 + c < D; c += 32) {
        const int col = h * D + c0 + c;
        const float g = a.proj[t * a.ldp + a.g_off + col], sg = sigmoid_f(g);
        const float v = o[c] * inv * a.onorm[col] * (DELTA ? sg : g * sg);
        if (f32) reinterpret_cast<float*>(a.out)[t * a.ldo + col] = v;
        else reinterpret_cast<__nv_bfloat16*>(a.out)[t * a.ldo + col] = __float2bfloat16(v);
      }
      __syncwarp();
    }
  };

  // ---- consumers: a column, and every fourth group of four key rows
  const int col = tid >> 2, kq = tid & 3, cg = c0 + col;
  float* sp = a.state + (size_t)row * a.row_stride + ((size_t)h * D + cg) * D;
  f2_t M[NQ * 2];
  if (consumer) {
    const bool mine = cg < D;
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int k = (kq + 4 * i) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (mine && (D & 3) == 0) {
        if (k < D) v = *reinterpret_cast<const float4*>(sp + k);
      } else if (mine) {
        if (k < D) v.x = sp[k];
        if (k + 1 < D) v.y = sp[k + 1];
        if (k + 2 < D) v.z = sp[k + 2];
        if (k + 3 < D) v.w = sp[k + 3];
      }
      M[2 * i] = pack2(v.x, v.y);
      M[2 * i + 1] = pack2(v.z, v.w);
    }
  } else if (n_tiles > 0) {
    stage(0);
  }
  barrier();
  const int last = CS > 1 ? n_tiles + 1 : n_tiles;
  for (int it = 0; it <= last; ++it) {
    if (!consumer) {
      if (it + 1 < n_tiles) stage(it + 1);
      if (CS == 1) {
        if (it >= 1) finish(it - 1, true);
      } else {
        if (it >= 1 && it - 1 < n_tiles) {
          const int n = min(TB, len - (it - 1) * TB);
          for (int tb = pw; tb < n; tb += SCAN_PRODUCERS) {
            const float q = square(obuf + (((it - 1) % 3) * TB + tb) * CC);
            if (lane == 0) ssq[((it - 1) & 1) * TB + tb] = q;
          }
        }
        if (it >= 2) finish(it - 2, false);
      }
    } else if (it < n_tiles) {
      const float* buf = scan_smem + (it & 1) * buf_floats;
      const float* val = buf + TB * NVEC * DKP;
      const float* scal = val + TB * CC;
      float* o_out = obuf + (it % 3) * TB * CC;
      const int n = min(TB, len - it * TB);
      for (int tb = 0; tb < n; ++tb) {
        const ulonglong2* dw = reinterpret_cast<const ulonglong2*>(buf + tb * DKP);
        const ulonglong2* dk = dw + TB * DKP / 4;
        const ulonglong2* dr = dk + TB * DKP / 4;
        const ulonglong2* du = dr + TB * DKP / 4;
        const ulonglong2* da = du + TB * DKP / 4;
        const float v = val[tb * CC + col], s2 = scal[2 * tb + 1];
        f2_t o2[2] = {0, 0}, g2[2] = {0, 0};
#pragma unroll
        for (int i = 0; i < NQ; ++i) {
          const ulonglong2 r = dr[kq + 4 * i];
          o2[0] = fma2(M[2 * i], r.x, o2[0]);
          o2[1] = fma2(M[2 * i + 1], r.y, o2[1]);
          if (DELTA) {
            const ulonglong2 u = du[kq + 4 * i];
            g2[0] = fma2(M[2 * i], u.x, g2[0]);
            g2[1] = fma2(M[2 * i + 1], u.y, g2[1]);
          }
        }
        float o = sum_of(o2[0]) + sum_of(o2[1]), gone = 0.f;
        if (DELTA) {
          gone = sum_of(g2[0]) + sum_of(g2[1]);
          gone += __shfl_xor_sync(0xffffffffu, gone, 1);
          gone += __shfl_xor_sync(0xffffffffu, gone, 2);
        }
        const f2_t vv = pack2(v, v), gg = pack2(-gone, -gone);
#pragma unroll
        for (int i = 0; i < NQ; ++i) {
          const ulonglong2 k = dk[kq + 4 * i], w = dw[kq + 4 * i];
          f2_t x = mul2(k.x, vv), y = mul2(k.y, vv);
          if (DELTA) {
            const ulonglong2 au = da[kq + 4 * i];
            x = fma2(au.x, gg, x);
            y = fma2(au.y, gg, y);
          }
          M[2 * i] = fma2(w.x, M[2 * i], x);
          M[2 * i + 1] = fma2(w.y, M[2 * i + 1], y);
        }
        o += __shfl_xor_sync(0xffffffffu, o, 1);
        o += __shfl_xor_sync(0xffffffffu, o, 2);
        if (kq == 0) o_out[tb * CC + col] = fmaf(s2, v, DELTA ? fmaf(-scal[2 * tb], gone, o) : o);
      }
    }
    barrier();
  }
  if (consumer && cg < D) {
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int k = (kq + 4 * i) * 4;
      const float2 lo = unpack2(M[2 * i]), hi = unpack2(M[2 * i + 1]);
      if ((D & 3) == 0) {
        if (k < D) *reinterpret_cast<float4*>(sp + k) = make_float4(lo.x, lo.y, hi.x, hi.y);
      } else {
        if (k < D) sp[k] = lo.x;
        if (k + 1 < D) sp[k + 1] = lo.y;
        if (k + 2 < D) sp[k + 2] = hi.x;
        if (k + 3 < D) sp[k + 3] = hi.y;
      }
    }
  }
}

template <typename AT>
__global__ void __launch_bounds__(128) tanh_rows_kernel(const float* x, int ldx, AT* out, int ldo, int n, int M, int pdl) {
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const long long all = (long long)M * n;
  for (long long i = (long long)blockIdx.x * 128 + threadIdx.x; i < all; i += (long long)gridDim.x * 128) {
    const int m = (int)(i / n), c = (int)(i - (long long)m * n);
    out[(size_t)m * ldo + c] = from_f32<AT>(tanhf(x[(size_t)m * ldx + c]));
  }
}

// Columns per CTA and CTAs per head: a head's columns are cut until the grid fills the machine (16 columns at the least); a
// CTA takes at most 128.
static void scan_split(int n_seq, int H, int D, int* CC, int* CS) {
  int cs = 1;
  while ((D + cs - 1) / cs > 128) cs *= 2;
  while (cs < 8 && (long long)n_seq * H * cs * 2 <= 148 && D / (cs * 2) >= 16) cs *= 2;
  const int cc = ((D + cs - 1) / cs + 7) / 8 * 8;
  *CC = cc;
  *CS = cs;
}

template <bool DELTA, int DKP>
static int scan_launch(const ScanArgs& a, int f32, cudaStream_t st) {
  int CC, CS;
  scan_split(a.r.n_seq, a.H, a.D, &CC, &CS);
  constexpr int TB = scan_tokens(DKP), NVEC = scan_vectors(DELTA);
  const int bytes = (2 * TB * (NVEC * DKP + CC + 2) + 3 * TB * CC + 2 * TB) * 4;
  CUDA_CHECK_RET(cudaFuncSetAttribute(scan_kernel<DELTA, DKP>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (CS > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = CS;
    attr[n].val.clusterDim.y = 1;
    attr[n].val.clusterDim.z = 1;
    ++n;
  }
  if (a.pdl) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(a.H * CS, a.r.n_seq);
  cfg.blockDim = dim3(CC * 4 + SCAN_PRODUCERS * 32);
  cfg.dynamicSmemBytes = bytes;
  cfg.stream = st;
  cfg.attrs = attr;
  cfg.numAttrs = n;
  CUDA_CHECK_RET(cudaLaunchKernelEx(&cfg, scan_kernel<DELTA, DKP>, a, CC, CS, f32));
  return 0;
}

template <bool DELTA>
static int scan_dispatch(const ScanArgs& a, int f32, cudaStream_t st) {
#define SMC_SCAN(N) if (a.D <= N) return scan_launch<DELTA, N>(a, f32, st);
  SMC_SCAN(16) SMC_SCAN(32) SMC_SCAN(48) SMC_SCAN(64) SMC_SCAN(80) SMC_SCAN(96) SMC_SCAN(128) SMC_SCAN(160) SMC_SCAN(192) SMC_SCAN(256)
#undef SMC_SCAN
  return -120;
}

}  // namespace smc

SMC_API int smc_scan_args_size() { return (int)sizeof(smc::ScanArgs); }

// One memory layer over the new tokens of every sequence; delta: the generalized delta rule, else the bonus form.  Heads of up
// to 256 columns.
SMC_API int smc_memory_scan(const smc::ScanArgs* a, int delta, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_seq <= 0) return 0;
  if (a->D < 1 || a->H < 1 || a->r.n_seq > 65535) return -120;
  return delta ? scan_dispatch<true>(*a, f32, st) : scan_dispatch<false>(*a, f32, st);
}

// out[m, c] = tanh(x[m, c]), c < n.
SMC_API int smc_tanh_rows(const float* x, int ldx, void* out, int ldo, int n, int M, int f32, int pdl, cudaStream_t st) {
  using namespace smc;
  if (M <= 0) return 0;
  const long long want = ((long long)M * n + 127) / 128;
  const dim3 grid((unsigned)(want < 2368 ? want : 2368)), block(128);
  if (f32) return launch_pdl(tanh_rows_kernel<float>, grid, block, 0, st, pdl, x, ldx, (float*)out, ldo, n, M, pdl);
  return launch_pdl(tanh_rows_kernel<__nv_bfloat16>, grid, block, 0, st, pdl, x, ldx, (__nv_bfloat16*)out, ldo, n, M, pdl);
}
