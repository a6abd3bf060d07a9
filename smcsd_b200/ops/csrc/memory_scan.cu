// Recurrent memories: one matrix [key, value] per head, advanced token by token in fp32.
//
//   delta   M <- diag(w) M - (a u)(u^T M) + k v^T, read out with r afterwards; u = k / |k|, a = sigmoid(. + bias),
//           w = exp(-log_decay sigmoid(z + w0)); output gate sigmoid
//   wkv     read out with r before the update, the current k v^T weighted by a bonus; M <- diag(w) M + k v^T,
//           w = exp(-exp(z + w0)); output gate silu
//   gated   M <- w M + a k v^T and a normaliser n <- w n + a k, read out with r afterwards and divided by
//           max(|n.r|, exp(-m)) + unit_eps; log gates i = cap tanh((. + bias) / cap), f = ln sigmoid(cap tanh(..)), running
//           maximum m <- max(f + m, i), w = exp(f + m_old - m), a = exp(i - m); output gate sigmoid.  The normaliser is one
//           more value column (of ones), which every CTA of a head keeps for itself.
//   channel M <- diag(w) M, then M <- M + b u (v - M^T u)^T, read out with r afterwards; u = k / |k|, r likewise times r_scale (both
//           shared by groups of heads), b = sigmoid(beta), w = exp(-exp(a_log) softplus(z + w0)); output gate sigmoid
//   forget  M <- diag(w) M + (1 - w) v^T, read out with silu(r) afterwards; w = lower + (1 - lower) sigmoid(. + bias); no output gate
// The elementwise functions of the last two are taken by a kernel of its own ahead of the scan, in place (scan_operands): the
// columns of a head are spread over CTAs, each of which would take them again, and the producers would not keep up.
//
// Value columns of a matrix never mix, key rows only in sums.  A CTA therefore keeps some columns of one head's matrix in
// registers - four or eight threads per pair of columns (one column beyond 128 key rows) share the key rows - and walks
// its sequence's tokens in tiles: consumer warps run the recurrence on the tile in shared memory while eight producer warps
// turn the next tile's projections into w, u, a u, ... and finish the outputs of the tile before (division by the head's root
// mean square, norm weight, gate).  Producers fetch a tile ahead of the one they prepare, so a tile's loads have a whole tile
// of consumer work to land in.  With few (sequence, head) pairs the columns of a head are spread over a thread-block cluster
// that exchanges the sums of squares through distributed shared memory.  Both sums over key rows are taken over the old
// matrix, so that a token costs one reduction: for delta the read-out is (r w)^T M - (r.a u)(u^T M) + (r.k) v, for channel, with g = (w u)^T M,
// (r w)^T M + (r.b u)(v - g).
// The recurrence is held to fp32 (a bf16 or tf32 chunk-parallel form would round the state), so the floor is the CUDA cores'
// rate; products and sums are issued two at a time (f32x2).
#include "memory_scan.cuh"

namespace smc {

constexpr int SCAN_PRODUCERS = 8;        // warps
constexpr int SCAN_CONSUMERS = 256;      // threads at the most
constexpr int SCAN_ALONE_BYTES = 118 * 1024;          // shared memory that leaves no room for a second CTA

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
// A store the compiler may move loads across: nobody reads the word before the next barrier.
__device__ __forceinline__ void store_shared_unordered(uint32_t addr, float v) {
  asm volatile("st.shared.f32 [%0], %1;" ::"r"(addr), "f"(v));
}
__device__ __forceinline__ float sum_of(f2_t a) { const float2 v = unpack2(a); return v.x + v.y; }

__host__ __device__ constexpr int scan_tokens(int dkp) { return dkp <= 128 ? 16 : 8; }       // tokens of a tile
__host__ __device__ constexpr int scan_vectors(int kind) { return kind == SCAN_DELTA ? 5 : kind == SCAN_CHANNEL ? 4 : kind == SCAN_GATED ? 2 : 3; }
__host__ __device__ constexpr int scan_columns(int dkp) { return dkp <= 128 ? 2 : 1; }       // of a consumer thread
// Consumer threads that share a column's key rows: eight give a token's chain half the length, at one more exchange per sum.
__host__ __device__ constexpr int scan_sharers(int kind, int dkp) {
  return (kind == SCAN_CHANNEL || kind == SCAN_FORGET) && dkp >= 64 && dkp <= 128 && dkp % 32 == 0 ? 8 : 4;
}
__host__ __device__ constexpr int scan_max_columns(int kind, int dkp) { return SCAN_CONSUMERS / scan_sharers(kind, dkp) * scan_columns(dkp); }      // of a CTA

template <int KIND, int DKP>
__global__ void __launch_bounds__(SCAN_CONSUMERS + SCAN_PRODUCERS * 32) scan_kernel(const ScanArgs a, int CC, int CS, int f32) {
  constexpr bool GENERAL = KIND == SCAN_DELTA, GATED = KIND == SCAN_GATED, CHANNEL = KIND == SCAN_CHANNEL, FORGET = KIND == SCAN_FORGET;
  constexpr bool DELTA = GENERAL || CHANNEL;                 // something is taken off along u
  constexpr bool SQUARE = GENERAL || KIND == SCAN_BONUS;     // as many values as keys
  constexpr int TB = scan_tokens(DKP), NVEC = scan_vectors(KIND), NL = (DKP + 31) / 32, CP = scan_columns(DKP);
  constexpr int KT = scan_sharers(KIND, DKP), NQ = DKP / (4 * KT), MOST = scan_max_columns(KIND, DKP);
  constexpr int PT = TB / SCAN_PRODUCERS;                    // tokens of a tile per producer warp
  constexpr int NC = ((!SQUARE || MOST < DKP ? MOST : DKP) + 31) / 32;      // columns of a CTA per lane
  extern __shared__ __align__(16) float scan_smem[];
  const int buf_floats = TB * (NVEC * DKP + CC + 2);
  float* obuf = scan_smem + 2 * buf_floats;                  // [3][TB][CC]
  float* ssq = obuf + 3 * TB * CC;                           // [2][TB]
  float* least = ssq + 2 * TB;                               // [4][TB] exp(-m) (gated)
  const int n_cons = CC / CP * KT, tid = threadIdx.x, lane = tid & 31;
  const bool consumer = tid < n_cons;
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int h = blockIdx.x / CS, rank = blockIdx.x - h * CS, s = blockIdx.y, D = a.D, V = a.V;
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
  const int own = GATED ? CC - 1 : CC;                       // value columns of this CTA; the last slot is the normaliser's
  const int n_tiles = (len + TB - 1) / TB, c0 = rank * own;
  const int last = CS > 1 ? n_tiles + 1 : n_tiles;

  if (!consumer) {
    const int pw = (tid - n_cons) >> 5;
    float kk[PT][NL], rr[PT][NL], zz[PT][NL], aa[PT][NL], vv[PT][NC], gg[PT][NC];
    float gi = 0.f, gf = 0.f, m_run = 0.f, bi = 0.f, bf = 0.f;       // gated: gate logits of token `lane` of a tile, running maximum
    float bb[PT];                                            // channel: write strengths
    const int hk = CHANNEL ? h / a.rep : h;
    if (GATED) {
      bi = a.a_bias[h];
      bf = a.a_bias[a.H + h];
      m_run = a.top[(size_t)row * a.row_stride + h];
    }
    auto fetch = [&](int tile) {                             // projections of a tile into registers
      const int n = min(TB, len - tile * TB);
#pragma unroll
      for (int j = 0; j < PT; ++j) {
        const int tb = pw + j * SCAN_PRODUCERS;
        const size_t t = (size_t)off + tile * TB + tb;
        const float* p = a.proj + t * a.ldp + hk * D;
        const float* pv = a.proj + t * a.ldp + h * V;
        const float* zr = a.z + t * a.ldz + h * D;
#pragma unroll
        for (int i = 0; i < NL; ++i) {
          const int c = lane + 32 * i;
          const bool ok = c < D && tb < n;
          if (!FORGET) kk[j][i] = ok ? p[a.k_off + c] : 0.f;
          rr[j][i] = ok ? p[a.r_off + c] : 0.f;
          if (!GATED && !FORGET) zz[j][i] = ok ? zr[c] : 0.f;
          if (GENERAL || FORGET) aa[j][i] = ok ? p[a.a_off + c] : 0.f;
        }
        if (CHANNEL) bb[j] = tb < n ? a.beta[t * a.ldb + h] : 0.f;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
          const int c = lane + 32 * i;
          vv[j][i] = c < own && c0 + c < V && tb < n ? pv[a.v_off + c0 + c] : 0.f;
        }
      }
      if (GATED && lane < n) {                               // every producer warp reads the gates of the whole tile
        const float* p = a.proj + ((size_t)off + tile * TB + lane) * a.ldp + a.a_off + h;
        gi = p[0];
        gf = p[a.H];
      }
    };
    auto stage = [&](int tile) {                             // registers to the consumers' operands
      float* buf = scan_smem + (tile & 1) * buf_floats;
      float* val = buf + TB * NVEC * DKP;
      float* scal = val + TB * CC;
      const int n = min(TB, len - tile * TB);
      float keep = 0.f, add = 0.f, low = 0.f;                // of token `lane`
      if (GATED) {
        // running maxima of a tile: a scan over pairs (sum of f, maximum), all in this warp
        const bool ok = lane < n;
        const float cap = a.gate_cap, li = ok ? cap * tanhf((gi + bi) / cap) : -INFINITY;
        const float lf = ok ? log_sigmoid_f(cap * tanhf((gf + bf) / cap)) : 0.f;
        float sum = lf, most = li;
#pragma unroll
        for (int o = 1; o < TB; o <<= 1) {
          const float s0 = __shfl_up_sync(0xffffffffu, sum, o), m0 = __shfl_up_sync(0xffffffffu, most, o);
          if (lane >= o) {
            most = fmaxf(most, m0 + sum);
            sum += s0;
          }
        }
        const float m = fmaxf(most, m_run + sum), up = __shfl_up_sync(0xffffffffu, m, 1), before = lane == 0 ? m_run : up;
        keep = expf(lf + before - m);
        add = expf(li - m);
        low = expf(-m);
        m_run = __shfl_sync(0xffffffffu, m, n - 1);
        if (pw == 0 && lane < n) least[(tile & 3) * TB + lane] = low;
      }
#pragma unroll
      for (int j = 0; j < PT; ++j) {
        const int tb = pw + j * SCAN_PRODUCERS;
        if (tb >= n) continue;
        float inv = 0.f, s1 = 0.f, s2 = 0.f, rinv = 0.f, b = 0.f;
        if (DELTA) {
          float ss = 0.f;
#pragma unroll
          for (int i = 0; i < NL; ++i) ss = fmaf(kk[j][i], kk[j][i], ss);
          inv = 1.0f / sqrtf(warp_sum(ss) + a.unit_eps);
        }
        if (CHANNEL) {
          float ss = 0.f;
#pragma unroll
          for (int i = 0; i < NL; ++i) ss = fmaf(rr[j][i], rr[j][i], ss);
          rinv = a.r_scale / sqrtf(warp_sum(ss) + a.unit_eps);
          b = sigmoid_f(bb[j]);
        }
        float* d = buf + tb * DKP;
#pragma unroll
        for (int i = 0; i < NL; ++i) {
          const int c = lane + 32 * i;
          if (c >= DKP) continue;
          const bool ok = c < D;
          if (GATED) {
            d[c] = kk[j][i];
            d[TB * DKP + c] = rr[j][i] * a.r_scale;
            s2 = fmaf(rr[j][i] * a.r_scale, kk[j][i], s2);
            continue;
          }
          if (CHANNEL) {
            const float w = zz[j][i], u = kk[j][i] * inv, r = rr[j][i] * rinv;
            d[c] = w;
            d[TB * DKP + c] = b * u;
            d[2 * TB * DKP + c] = r * w;
            d[3 * TB * DKP + c] = w * u;
            s2 = fmaf(r, b * u, s2);
            continue;
          }
          if (FORGET) {
            const float k = aa[j][i], w = ok ? 1.0f - k : 0.f, r = rr[j][i];
            d[c] = w;
            d[TB * DKP + c] = k;
            d[2 * TB * DKP + c] = r * w;
            s2 = fmaf(r, k, s2);
            continue;
          }
          const float z = ok ? zz[j][i] + a.w0[h * D + c] : 0.f;
          const float w = !ok ? 0.f : DELTA ? expf(-a.log_decay * sigmoid_f(z)) : expf(-expf(z));
          d[c] = w;
          d[TB * DKP + c] = kk[j][i];
          if (DELTA) {
            const float u = kk[j][i] * inv, au = ok ? sigmoid_f(aa[j][i] + a.a_bias[h * D + c]) * u : 0.f;
            d[2 * TB * DKP + c] = rr[j][i] * w;
            d[3 * TB * DKP + c] = u;
            d[(NVEC - 1) * TB * DKP + c] = au;
            s1 = fmaf(rr[j][i], au, s1);
            s2 = fmaf(rr[j][i], kk[j][i], s2);
          } else {
            d[2 * TB * DKP + c] = rr[j][i];
            s2 = fmaf(rr[j][i] * (ok ? a.bonus[h * D + c] : 0.f), kk[j][i], s2);
          }
        }
#pragma unroll
        for (int i = 0; i < NC; ++i)
          if (lane + 32 * i < CC) val[tb * CC + lane + 32 * i] = vv[j][i];
        if (GATED) {
          const float w = __shfl_sync(0xffffffffu, add, tb);
#pragma unroll
          for (int i = 0; i < NC; ++i)
            if (lane + 32 * i < CC) val[tb * CC + lane + 32 * i] = lane + 32 * i < own ? w * vv[j][i] : w;
        }
        __syncwarp();
        s1 = GENERAL ? warp_sum(s1) : GATED ? __shfl_sync(0xffffffffu, keep, tb) : 0.f;
        s2 = warp_sum(s2);
        if (lane == 0) { scal[2 * tb] = s1; scal[2 * tb + 1] = s2; }
      }
    };
    auto gates = [&](int tile) {                             // gate columns of a tile into registers
      const int n = min(TB, len - tile * TB);
#pragma unroll
      for (int j = 0; j < PT; ++j) {
        const int tb = pw + j * SCAN_PRODUCERS;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
          const int c = lane + 32 * i;
          const size_t t = (size_t)off + tile * TB + tb;
          const float* g = CHANNEL ? a.gate + t * a.ldg : a.proj + t * a.ldp + a.g_off;
          gg[j][i] = !FORGET && c < own && c0 + c < V && tb < n ? g[h * V + c0 + c] : 0.f;
        }
      }
    };
    auto square = [&](const float* o) {
      float q = 0.f;
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const float v = lane + 32 * i < own ? o[lane + 32 * i] : 0.f;      // columns beyond V are zero
        q = fmaf(v, v, q);
      }
      return warp_sum(q);
    };
    auto finish = [&](int tile) {
      const int n = min(TB, len - tile * TB);
#pragma unroll
      for (int j = 0; j < PT; ++j) {
        const int tb = pw + j * SCAN_PRODUCERS;
        if (tb >= n) continue;
        const size_t t = (size_t)off + tile * TB + tb;
        const float* o = obuf + ((tile % 3) * TB + tb) * CC;
        float tot = 0.f;
        if (CS == 1) {
          tot = square(o);
        } else {
          const uint32_t at = smem_u32(ssq + (tile & 1) * TB + tb);
          for (int q = 0; q < CS; ++q) tot += ld_dsmem_f32(at, q);
        }
        float unit = 1.0f;                                   // gated: the read-out's divisor
        if (GATED) unit = 1.0f / (fmaxf(fabsf(o[CC - 1]), least[(tile & 3) * TB + tb]) + a.unit_eps);
        const float inv = unit / sqrtf(tot * unit * unit / (float)V + a.eps);
#pragma unroll
        for (int i = 0; i < NC; ++i) {
          const int c = lane + 32 * i, col = h * V + c0 + c;
          if (c >= own || c0 + c >= V) continue;
          const float g = gg[j][i], sg = CHANNEL || FORGET ? 1.0f : sigmoid_f(g);
          const float v = o[c] * inv * (CHANNEL ? g : a.onorm[col] * (FORGET || GENERAL || GATED ? sg : g * sg));
          if (f32) reinterpret_cast<float*>(a.out)[t * a.ldo + col] = v;
          else reinterpret_cast<__nv_bfloat16*>(a.out)[t * a.ldo + col] = __float2bfloat16(v);
        }
        __syncwarp();
      }
    };
    const int lag = CS > 1 ? 2 : 1;                          // tiles between a tile's recurrence and its outputs
    if (n_tiles > 0) {
      fetch(0);
      stage(0);
      if (n_tiles > 1) fetch(1);
      if (lag == 1) gates(0);
    }
    barrier();
    for (int it = 0; it <= last; ++it) {
      if (it + 1 < n_tiles) stage(it + 1);
      if (it + 2 < n_tiles) fetch(it + 2);
      if (CS > 1 && it >= 1 && it - 1 < n_tiles) {
        const int n = min(TB, len - (it - 1) * TB);
        for (int tb = pw; tb < n; tb += SCAN_PRODUCERS) {
          const float q = square(obuf + (((it - 1) % 3) * TB + tb) * CC);
          if (lane == 0) ssq[((it - 1) & 1) * TB + tb] = q;
        }
      }
      if (it >= lag) finish(it - lag);
      const int next = it + 1 - lag;                         // the tile the next round finishes
      if (next >= 0 && next < n_tiles && (lag > 1 || it > 0)) gates(next);
      barrier();
    }
    if (GATED && rank == 0 && pw == 0 && lane == 0) a.top[(size_t)row * a.row_stride + h] = m_run;
    return;
  }

  // ---- consumers: CP columns, and every KT-th group of four key rows
  const int col = tid / KT * CP, kq = tid % KT;
  auto column = [&](int x) {                                 // row of the transposed matrix (-1: none)
    if (GATED && col + x == CC - 1) return V;
    return col + x < own && c0 + col + x < V ? c0 + col + x : -1;
  };
  f2_t M[CP][NQ * 2];
  float* sp[CP];
#pragma unroll
  for (int x = 0; x < CP; ++x) {
    const int cg = column(x);
    const bool mine = cg >= 0;
    sp[x] = a.state + (size_t)row * a.row_stride + ((size_t)h * (V + GATED) + (mine ? cg : 0)) * D;
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int k = (kq + KT * i) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (mine && (D & 3) == 0) {
        if (k < D) v = *reinterpret_cast<const float4*>(sp[x] + k);
      } else if (mine) {
        if (k < D) v.x = sp[x][k];
        if (k + 1 < D) v.y = sp[x][k + 1];
        if (k + 2 < D) v.z = sp[x][k + 2];
        if (k + 3 < D) v.w = sp[x][k + 3];
      }
      M[x][2 * i] = pack2(v.x, v.y);
      M[x][2 * i + 1] = pack2(v.z, v.w);
    }
  }
  barrier();
  for (int it = 0; it <= last; ++it) {
    if (it < n_tiles) {
      const float* buf = scan_smem + (it & 1) * buf_floats;
      const float* val = buf + TB * NVEC * DKP;
      const float* scal = val + TB * CC;
      const uint32_t o_out = smem_u32(obuf + (it % 3) * TB * CC);
      const int n = min(TB, len - it * TB);
#pragma unroll 2
      for (int tb = 0; tb < n; ++tb) {
        const ulonglong2* dw = reinterpret_cast<const ulonglong2*>(buf + tb * DKP);
        const ulonglong2* dk = GATED ? dw : dw + TB * DKP / 4;
        const ulonglong2* dr = dk + TB * DKP / 4;
        const ulonglong2* du = dr + TB * DKP / 4;
        const ulonglong2* da = du + TB * DKP / 4;
        const float s1 = scal[2 * tb], s2 = scal[2 * tb + 1];
        float v[CP];
        f2_t o2[CP][2], g2[CP][2];
#pragma unroll
        for (int x = 0; x < CP; ++x) {
          v[x] = val[tb * CC + col + x];
          o2[x][0] = o2[x][1] = g2[x][0] = g2[x][1] = 0;
        }
#pragma unroll
        for (int i = 0; i < NQ; ++i) {
          if (DELTA) {
            const ulonglong2 u = du[kq + KT * i];
#pragma unroll
            for (int x = 0; x < CP; ++x) {
              g2[x][0] = fma2(M[x][2 * i], u.x, g2[x][0]);
              g2[x][1] = fma2(M[x][2 * i + 1], u.y, g2[x][1]);
            }
          }
        }
        float o[CP], gone[CP];
#pragma unroll
        for (int x = 0; x < CP; ++x) {
          gone[x] = 0.f;
          if (DELTA) {
            gone[x] = sum_of(g2[x][0]) + sum_of(g2[x][1]);
#pragma unroll
            for (int s = 1; s < KT; s <<= 1) gone[x] += __shfl_xor_sync(0xffffffffu, gone[x], s);
          }
        }
#pragma unroll
        for (int i = 0; i < NQ; ++i) {
          const ulonglong2 r = dr[kq + KT * i];
#pragma unroll
          for (int x = 0; x < CP; ++x) {
            o2[x][0] = fma2(M[x][2 * i], r.x, o2[x][0]);
            o2[x][1] = fma2(M[x][2 * i + 1], r.y, o2[x][1]);
          }
        }
        f2_t vv[CP], gg[CP];
#pragma unroll
        for (int x = 0; x < CP; ++x) {
          o[x] = sum_of(o2[x][0]) + sum_of(o2[x][1]);
          if (CHANNEL) v[x] -= gone[x];
          vv[x] = pack2(v[x], v[x]);
          gg[x] = pack2(-gone[x], -gone[x]);
        }
#pragma unroll
        for (int i = 0; i < NQ; ++i) {
          const ulonglong2 k = dk[kq + KT * i];
          ulonglong2 w;
          if (GATED) w.x = w.y = pack2(s1, s1); else w = dw[kq + KT * i];
          ulonglong2 au;
          if (GENERAL) au = da[kq + KT * i];
#pragma unroll
          for (int x = 0; x < CP; ++x) {
            f2_t p = mul2(k.x, vv[x]), q = mul2(k.y, vv[x]);
            if (GENERAL) {
              p = fma2(au.x, gg[x], p);
              q = fma2(au.y, gg[x], q);
            }
            M[x][2 * i] = fma2(w.x, M[x][2 * i], p);
            M[x][2 * i + 1] = fma2(w.y, M[x][2 * i + 1], q);
          }
        }
#pragma unroll
        for (int x = 0; x < CP; ++x) {
#pragma unroll
          for (int s = 1; s < KT; s <<= 1) o[x] += __shfl_xor_sync(0xffffffffu, o[x], s);
          if (kq == 0)
            store_shared_unordered(o_out + (tb * CC + col + x) * 4, fmaf(s2, v[x], GENERAL ? fmaf(-s1, gone[x], o[x]) : GATED ? s1 * o[x] : o[x]));
        }
      }
    }
    barrier();
  }
#pragma unroll
  for (int x = 0; x < CP; ++x) {
    if (column(x) < 0 || (GATED && column(x) == V && rank != 0)) continue;
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int k = (kq + KT * i) * 4;
      const float2 lo = unpack2(M[x][2 * i]), hi = unpack2(M[x][2 * i + 1]);
      if ((D & 3) == 0) {
        if (k < D) *reinterpret_cast<float4*>(sp[x] + k) = make_float4(lo.x, lo.y, hi.x, hi.y);
      } else {
        if (k < D) sp[x][k] = lo.x;
        if (k + 1 < D) sp[x][k + 1] = lo.y;
        if (k + 2 < D) sp[x][k + 2] = hi.x;
        if (k + 3 < D) sp[x][k + 3] = hi.y;
      }
    }
  }
}

// Elementwise operands of the kinds channel and forget, in place, four (or one) columns per thread:
//   channel  z <- exp(-exp(a_log) softplus(z + w0)), gate <- sigmoid(gate) onorm
//   forget   r <- silu(r), forget gate <- 1 - w = (1 - lower) sigmoid(-(. + bias)): what is written keeps its relative accuracy
template <int KIND, int VEC>
__global__ void __launch_bounds__(128) scan_operands_kernel(const ScanArgs a, int T) {
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int HD = a.H * a.D, n2 = KIND == SCAN_CHANNEL ? a.H * a.V : HD, c = (blockIdx.x * 128 + threadIdx.x) * VEC;
  if (c >= HD + n2) return;
  const bool second = c >= HD;                               // VEC divides HD
  const int at = second ? c - HD : c;
  float w[VEC], l[VEC];
#pragma unroll
  for (int k = 0; k < VEC; ++k) {
    w[k] = KIND == SCAN_CHANNEL ? (second ? a.onorm[at + k] : a.w0[at + k]) : a.a_bias[at + k];
    l[k] = KIND == SCAN_CHANNEL ? (second ? 0.f : -expf(a.a_log[(at + k) / a.D])) : 1.0f - a.lower[at + k];
  }
  for (int t = blockIdx.y; t < T; t += gridDim.y) {
    float* p = const_cast<float*>(KIND == SCAN_CHANNEL ? (second ? a.gate + (size_t)t * a.ldg : a.z + (size_t)t * a.ldz)
                                                       : a.proj + (size_t)t * a.ldp + (second ? a.a_off : a.r_off)) + at;
    float v[VEC];
    load_cols<VEC>(v, (const float*)p);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
      if (KIND == SCAN_CHANNEL) v[k] = second ? sigmoid_f(v[k]) * w[k] : expf(l[k] * softplus_f(v[k] + w[k]));
      else v[k] = second ? l[k] * sigmoid_f(-(v[k] + w[k])) : v[k] * sigmoid_f(v[k]);
    }
    store_cols<VEC>(p, v);
  }
}

template <int KIND>
static int scan_operands(const ScanArgs& a, int T, cudaStream_t st) {
  const int HD = a.H * a.D, n = HD + (KIND == SCAN_CHANNEL ? a.H * a.V : HD);
  const bool vec = HD % 4 == 0 && n % 4 == 0 && a.D % 4 == 0 &&
                   (KIND == SCAN_CHANNEL ? a.ldz % 4 == 0 && a.ldg % 4 == 0 : (a.ldp | a.r_off | a.a_off) % 4 == 0);
  const dim3 grid((n / (vec ? 4 : 1) + 127) / 128, T < 1024 ? T : 1024), block(128);
  return vec ? launch_pdl(scan_operands_kernel<KIND, 4>, grid, block, 0, st, a.pdl, a, T)
             : launch_pdl(scan_operands_kernel<KIND, 1>, grid, block, 0, st, a.pdl, a, T);
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

// Decay logits of few tokens in one launch: z[t, n] = sum_k W[n, k] tanh(x[t, k]), tanh rounded to the activation type as the
// GEMM's operand would be; a thread per output.
template <typename AT>
__global__ void __launch_bounds__(64) low_rank_kernel(const float* x, int ldx, const AT* W, float* z, int ldz, int N, int K, int pdl) {
  extern __shared__ __align__(16) float lr_smem[];
  const int n = blockIdx.x * 64 + threadIdx.x, t = blockIdx.y;
  const AT* w = W + (size_t)min(n, N - 1) * K;
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  for (int k = threadIdx.x; k < K; k += 64) lr_smem[k] = to_f32<AT>(from_f32<AT>(tanhf(x[(size_t)t * ldx + k])));
  __syncthreads();
  float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
  for (int k = 0; k < K; k += 4) {
    const float4 a = load4(w + k), b = load4((const float*)lr_smem + k);
    s[0] = fmaf(a.x, b.x, s[0]);
    s[1] = fmaf(a.y, b.y, s[1]);
    s[2] = fmaf(a.z, b.z, s[2]);
    s[3] = fmaf(a.w, b.w, s[3]);
  }
  if (n < N) z[(size_t)t * ldz + n] = (s[0] + s[1]) + (s[2] + s[3]);
}

// Columns per CTA and CTAs per head: a head's columns are cut until the grid fills the machine (16 columns at the least); a
// CTA takes at most scan_max_columns, `extra` of them beside its share of the head's.  Whole warps of consumers need multiples
// of 8 (16 in pairs), half of that with eight threads per pair.
static void scan_split(int n_seq, int H, int V, int most, int unit, int extra, int* CC, int* CS) {
  int cs = 1;
  while ((V + cs - 1) / cs + extra > most) cs *= 2;
  while (cs < 8 && (long long)n_seq * H * cs * 2 <= 148 && V / (cs * 2) >= 16) cs *= 2;
  *CC = ((V + cs - 1) / cs + extra + unit - 1) / unit * unit;
  *CS = cs;
}

template <int KIND, int DKP>
static int scan_launch(const ScanArgs& a, int f32, cudaStream_t st) {
  int CC, CS;
  constexpr int TB = scan_tokens(DKP), NVEC = scan_vectors(KIND), CP = scan_columns(DKP), KT = scan_sharers(KIND, DKP);
  scan_split(a.r.n_seq, a.H, a.V, scan_max_columns(KIND, DKP), 32 / KT * CP, KIND == SCAN_GATED, &CC, &CS);
  if (CS > 16) return -122;
  int bytes = (2 * TB * (NVEC * DKP + CC + 2) + 3 * TB * CC + 6 * TB) * 4;
  // a grid of no more CTAs than SMs: one each, also where the launch overlaps the kernel before and SMs are unevenly free
  if ((KIND == SCAN_CHANNEL || KIND == SCAN_FORGET) && (long long)a.H * CS * a.r.n_seq <= 148 && bytes < SCAN_ALONE_BYTES) bytes = SCAN_ALONE_BYTES;
  CUDA_CHECK_RET(cudaFuncSetAttribute(scan_kernel<KIND, DKP>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
  if (CS > 8) CUDA_CHECK_RET(cudaFuncSetAttribute(scan_kernel<KIND, DKP>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
  return launch_cluster(scan_kernel<KIND, DKP>, dim3(a.H * CS, a.r.n_seq), dim3(CC / CP * KT + SCAN_PRODUCERS * 32), bytes, st, a.pdl,
                        CS, a, CC, CS, f32);
}

template <int KIND>
static int scan_dispatch(const ScanArgs& a, int f32, cudaStream_t st) {
#define SMC_SCAN(N) if (a.D <= N) return scan_launch<KIND, N>(a, f32, st);
  SMC_SCAN(16) SMC_SCAN(32) SMC_SCAN(48) SMC_SCAN(64) SMC_SCAN(80) SMC_SCAN(96) SMC_SCAN(128) SMC_SCAN(160) SMC_SCAN(192) SMC_SCAN(256)
#undef SMC_SCAN
  return -120;
}

}  // namespace smc

SMC_API int smc_scan_args_size() { return (int)sizeof(smc::ScanArgs); }

// One memory layer over the new tokens of every sequence; kind: 0 the bonus form, 1 the generalized delta rule (both V = D), 2
// the gated form, 3 the delta rule with a decay per channel, 4 the forget-gated form (the last two overwrite their operands, T
// rows in all).  Heads of up to 256 key columns.
SMC_API int smc_memory_scan(const smc::ScanArgs* a, int kind, int T, int f32, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_seq <= 0) return 0;
  if (a->D < 1 || a->H < 1 || a->V < 1 || a->r.n_seq > 65535 || (kind < SCAN_GATED && a->V != a->D)) return -120;
  if (kind == SCAN_CHANNEL && (a->rep < 1 || a->H % a->rep)) return -120;
  switch (kind) {
    case SCAN_BONUS: return scan_dispatch<SCAN_BONUS>(*a, f32, st);
    case SCAN_DELTA: return scan_dispatch<SCAN_DELTA>(*a, f32, st);
    case SCAN_GATED: return scan_dispatch<SCAN_GATED>(*a, f32, st);
    case SCAN_CHANNEL:
      if (const int rc = scan_operands<SCAN_CHANNEL>(*a, T, st)) return rc;
      return scan_dispatch<SCAN_CHANNEL>(*a, f32, st);
    case SCAN_FORGET:
      if (const int rc = scan_operands<SCAN_FORGET>(*a, T, st)) return rc;
      return scan_dispatch<SCAN_FORGET>(*a, f32, st);
  }
  return -120;
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

// z = tanh(x) W^T for a few tokens; W [N, K], K a multiple of 8.
SMC_API int smc_low_rank(const float* x, int ldx, const void* W, float* z, int ldz, int N, int K, int M, int f32, int pdl,
                         cudaStream_t st) {
  using namespace smc;
  if (M <= 0) return 0;
  if (K % 8 || K > 8192 || M > 65535) return -121;
  const dim3 grid((N + 63) / 64, M), block(64);
  if (f32) return launch_pdl(low_rank_kernel<float>, grid, block, K * 4, st, pdl, x, ldx, (const float*)W, z, ldz, N, K, pdl);
  return launch_pdl(low_rank_kernel<__nv_bfloat16>, grid, block, K * 4, st, pdl, x, ldx, (const __nv_bfloat16*)W, z, ldz, N, K, pdl);
}
