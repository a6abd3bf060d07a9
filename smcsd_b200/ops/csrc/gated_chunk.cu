// The gated memory of memory_scan.cu for prompts in bf16, 64 tokens at a time on the tensor cores.
//
// With b the running sum of the log forget gates inside a chunk, m the running maxima and S, n, m0 what the chunk starts from:
//   read-out   S_t^T q_t = exp(b_t + m0 - m_t) S^T q_t + sum_{s <= t} exp(b_t - b_s + i_s - m_t) (k_s . q_t) v_s
//   state      S' = exp(b_L + m0 - m_L) S + sum_s k_s (exp(b_L - b_s + i_s - m_L) v_s)^T
// and the normaliser is one more value column of ones.  A CTA takes 64 value columns (and the normaliser) of one head, the CTAs of
// a head are a cluster that exchanges the rows' sums of squares.  The state lives in fp32 accumulator registers, and
// every operand of a product is two bf16 parts (hi + lo, about 2^-17; lo lo is left out): a read-out that is small is a difference
// of large terms, and the norm behind it brings their rounding up.  Gates, exponentials, maxima, divisors and norms are fp32.  The chain from
// chunk to chunk is short products of fragments that stay in registers, which the warp-level mma.sync serves without a trip
// through tensor memory per chunk.
#include "memory_scan.cuh"
#include "mma_sync.cuh"

namespace smc {

constexpr int GC_L = 64;                         // tokens of a chunk
constexpr int GC_EV = 64;                        // value columns of a CTA
constexpr int GC_LV = GC_EV + 8;                 // row pitch of value tiles: the columns, the normaliser's, seven of zeros
constexpr int GC_NT = GC_LV / 8;                 // column tiles
constexpr int GC_THREADS = 256;

__device__ __forceinline__ float gc_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gc_sigmoid(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }      // of the output gate

template <int DKP> struct GcShared {
  float q[GC_L][DKP], k[GC_L][DKP], v[GC_L][GC_EV];                      // as they come from the projection
  __nv_bfloat16 bq[2][GC_L][DKP + 8], bk[2][GC_L][DKP + 8];              // hi, lo
  __nv_bfloat16 bv[2][GC_L][GC_LV], wv_hi[GC_L][GC_LV], wv_lo[GC_L][GC_LV];
  __nv_bfloat16 s_hi[DKP][GC_LV], s_lo[DKP][GC_LV];
  float A[GC_L], B[GC_L], carry[GC_L], low[GC_L], w[GC_L];               // A, B in units of ln 2
  float decay, part[2][GC_L], ssq[2][GC_L];
};

template <int DKP>
__global__ void __launch_bounds__(GC_THREADS, 1) gated_chunk_kernel(const ScanArgs a, int CS) {
  constexpr int KD = DKP / 16, GROUPS = 128 / DKP, NTW = (GC_NT + GROUPS - 1) / GROUPS;
  constexpr float LOG2E = 1.4426950408889634f;
  extern __shared__ __align__(16) uint8_t gc_smem[];
  GcShared<DKP>& S = *reinterpret_cast<GcShared<DKP>*>(gc_smem);
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const int h = blockIdx.x / CS, rank = blockIdx.x - h * CS, s = blockIdx.y, D = a.D, V = a.V, H = a.H;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c0 = rank * GC_EV, nv = min(GC_EV, V - c0);
  const int row = a.r.seq_row[s];
  const int off = a.r.seq_off != nullptr ? a.r.seq_off[s] : s * a.r.E, len = a.r.seq_len != nullptr ? a.r.seq_len[s] : a.r.E;
  if (row < 0 || row >= a.n_rows) {              // the same in every CTA of the cluster
    if (tid == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  if (len <= 0) return;
  const int n_chunks = (len + GC_L - 1) / GC_L;
  float* M = a.state + (size_t)row * a.row_stride + (size_t)h * (V + 1) * D;
  float* top = a.top + (size_t)row * a.row_stride + h;

  // ---- fetching
  auto fetch = [&](int chunk) {
    const int n = min(GC_L, len - chunk * GC_L);
    const float* p = a.proj + ((size_t)off + chunk * GC_L) * a.ldp;
    for (int x = tid; x < GC_L * DKP / 4; x += GC_THREADS) {
      const int t = x / (DKP / 4), c = (x - t * (DKP / 4)) * 4;
      const bool real = t < n && c < D;
      const float* src = p + (real ? (size_t)t * a.ldp + h * D + c : 0);
      cp_async16(smem_u32(&S.q[t][c]), src + (real ? a.r_off : 0), real);
      cp_async16(smem_u32(&S.k[t][c]), src + (real ? a.k_off : 0), real);
    }
    for (int x = tid; x < GC_L * GC_EV / 4; x += GC_THREADS) {
      const int t = x / (GC_EV / 4), c = (x - t * (GC_EV / 4)) * 4;
      const bool real = t < n && c < nv;
      cp_async16(smem_u32(&S.v[t][c]), p + (real ? (size_t)t * a.ldp + a.v_off + h * V + c0 + c : 0), real);
    }
    cp_async_commit();
  };
  float gi[2] = {0.f, 0.f}, gf[2] = {0.f, 0.f};  // warp 0: gate logits of tokens 2 lane and 2 lane + 1 of the next chunk
  auto fetch_gates = [&](int chunk) {
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int t = chunk * GC_L + 2 * lane + j;
      if (t < len) {
        const float* p = a.proj + ((size_t)off + t) * a.ldp + a.a_off + h;
        gi[j] = p[0];
        gf[j] = p[H];
      }
    }
  };
  fetch(0);
  float m_run = 0.f, bias_i = 0.f, bias_f = 0.f;
  if (warp == 0) {
    m_run = *top;
    bias_i = a.a_bias[h];
    bias_f = a.a_bias[H + h];
    fetch_gates(0);
  }

  // ---- state: this warp's 16 key rows, NTW column tiles
  const int strip = warp % KD, tile0 = KD >= 8 ? 0 : (warp / KD) * NTW;
  float st[NTW][4];
  auto state_at = [&](int j, int e, bool& real) {            // element e of tile j: where it lives
    const int kr = strip * 16 + (lane >> 2) + (e >> 1) * 8, c = (tile0 + j) * 8 + (lane & 3) * 2 + (e & 1);
    real = kr < D && tile0 + j < GC_NT && (c < nv || c == GC_EV);
    return (size_t)(c == GC_EV ? V : c0 + c) * D + kr;
  };
  auto publish = [&]() {                                     // the state as operands
#pragma unroll
    for (int j = 0; j < NTW; ++j) {
      if (tile0 + j >= GC_NT) continue;
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int kr = strip * 16 + (lane >> 2) + r * 8, c = (tile0 + j) * 8 + (lane & 3) * 2;
        uint32_t hi, lo;
        split_bf16(st[j][2 * r], st[j][2 * r + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(&S.s_hi[kr][c]) = hi;
        *reinterpret_cast<uint32_t*>(&S.s_lo[kr][c]) = lo;
      }
    }
  };
#pragma unroll
  for (int j = 0; j < NTW; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      bool real;
      const size_t at = state_at(j, e, real);
      st[j][e] = real ? M[at] : 0.f;
    }
  publish();

  // ---- read-out: this warp's 16 tokens, half of the columns and the normaliser's tile
  const int half = warp >> 2, rs = half ? 3 - (warp & 3) : warp & 3;     // heavy and light token strips share a scheduler
  const int r0 = rs * 16 + (lane >> 2);                      // this thread's tokens: r0 and r0 + 8
  const uint32_t q_addr = smem_u32(&S.bq[0][rs * 16 + (lane & 15)][(lane >> 4) * 8]);
  const uint32_t k_addr = smem_u32(&S.bk[0][(lane & 7) + ((lane >> 4) << 3)][((lane >> 3) & 1) * 8]);
  const uint32_t v_addr = smem_u32(&S.bv[0][lane & 15][half * 32 + (lane >> 4) * 8]), v1_addr = smem_u32(&S.bv[0][lane & 15][GC_EV]);
  const uint32_t s_addr = smem_u32(&S.s_hi[lane & 15][half * 32 + (lane >> 4) * 8]), s1_addr = smem_u32(&S.s_hi[lane & 15][GC_EV]);
  constexpr uint32_t S_LO = sizeof(S.s_hi), WV_LO = sizeof(S.wv_hi), QK_LO = sizeof(S.bq[0]);
  const uint32_t kt_addr = smem_u32(&S.bk[0][(lane & 7) + ((lane >> 4) & 1) * 8][strip * 16 + ((lane >> 3) & 1) * 8]);
  const uint32_t wv_addr = smem_u32(&S.wv_hi[lane & 15][0]);

  for (int ch = 0; ch < n_chunks; ++ch) {
    const int n = min(GC_L, len - ch * GC_L);
    cp_async_wait<0>();
    __syncthreads();
    if (warp == 0) {
      // running sums and maxima of the chunk: a scan over pairs (sum of f, maximum), two tokens per lane
      const float cap = a.gate_cap;
      float li[2], lf[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const bool ok = 2 * lane + j < n;
        li[j] = ok ? cap * tanhf((gi[j] + bias_i) / cap) : -INFINITY;
        lf[j] = ok ? log_sigmoid_f(cap * tanhf((gf[j] + bias_f) / cap)) : 0.f;
      }
      float sum = lf[0] + lf[1], most = fmaxf(li[1], li[0] + lf[1]);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float s0 = __shfl_up_sync(0xffffffffu, sum, o), m0 = __shfl_up_sync(0xffffffffu, most, o);
        if (lane >= o) {
          most = fmaxf(most, m0 + sum);
          sum += s0;
        }
      }
      float b = __shfl_up_sync(0xffffffffu, sum, 1), m = __shfl_up_sync(0xffffffffu, most, 1);
      if (lane == 0) { b = 0.f; m = -INFINITY; }
      m = fmaxf(m, m_run + b);
      float A[2], B[2], mt[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        b += lf[j];
        m = fmaxf(m + lf[j], li[j]);
        A[j] = b - m;
        B[j] = li[j] - b;
        mt[j] = m;
      }
      const float a_end = __shfl_sync(0xffffffffu, A[1], 31), m_end = __shfl_sync(0xffffffffu, mt[1], 31);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = 2 * lane + j;
        S.A[t] = A[j] * LOG2E;
        S.B[t] = B[j] * LOG2E;
        S.carry[t] = expf(A[j] + m_run);
        S.low[t] = expf(-mt[j]);
        S.w[t] = expf(B[j] + a_end);
      }
      if (lane == 0) S.decay = expf(a_end + m_run);
      m_run = m_end;
      if (ch + 1 < n_chunks) fetch_gates(ch + 1);
    } else {
      for (int x = tid - 32; x < GC_L * DKP / 4; x += GC_THREADS - 32) {
        const int t = x / (DKP / 4), c = (x - t * (DKP / 4)) * 4;
        const float4 q = load4((const float*)&S.q[t][c]), k = load4((const float*)&S.k[t][c]);
        uint2 hi, lo;
        split_bf16(q.x * a.r_scale, q.y * a.r_scale, hi.x, lo.x);
        split_bf16(q.z * a.r_scale, q.w * a.r_scale, hi.y, lo.y);
        *reinterpret_cast<uint2*>(&S.bq[0][t][c]) = hi;
        *reinterpret_cast<uint2*>(&S.bq[1][t][c]) = lo;
        split_bf16(k.x, k.y, hi.x, lo.x);
        split_bf16(k.z, k.w, hi.y, lo.y);
        *reinterpret_cast<uint2*>(&S.bk[0][t][c]) = hi;
        *reinterpret_cast<uint2*>(&S.bk[1][t][c]) = lo;
      }
    }
    __syncthreads();
    for (int x = tid; x < GC_L * GC_LV / 4; x += GC_THREADS) {
      const int t = x / (GC_LV / 4), c = (x - t * (GC_LV / 4)) * 4;
      float4 v = make_float4(c == GC_EV && t < n ? 1.f : 0.f, 0.f, 0.f, 0.f);
      if (c < GC_EV) v = load4((const float*)&S.v[t][c]);
      const float w = S.w[t];
      uint2 hi, lo;
      split_bf16(v.x, v.y, hi.x, lo.x);
      split_bf16(v.z, v.w, hi.y, lo.y);
      *reinterpret_cast<uint2*>(&S.bv[0][t][c]) = hi;
      *reinterpret_cast<uint2*>(&S.bv[1][t][c]) = lo;
      split_bf16(w * v.x, w * v.y, hi.x, lo.x);
      split_bf16(w * v.z, w * v.w, hi.y, lo.y);
      *reinterpret_cast<uint2*>(&S.wv_hi[t][c]) = hi;
      *reinterpret_cast<uint2*>(&S.wv_lo[t][c]) = lo;
    }
    __syncthreads();
    if (ch + 1 < n_chunks) fetch(ch + 1);

    // ---- read-out
    float acc[5][4];
#pragma unroll
    for (int j = 0; j < 5; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
    float sc[GC_L / 16][2][4];                               // scores against 16 tokens at a time, up to the diagonal
#pragma unroll
    for (int kk = 0; kk < GC_L / 16; ++kk)
#pragma unroll
      for (int e = 0; e < 8; ++e) sc[kk][e >> 2][e & 3] = 0.f;
#pragma unroll 2
    for (int kd = 0; kd < KD; ++kd) {
      uint32_t qh[4], ql[4];
      ldsm4(qh, q_addr + kd * 32);
      ldsm4(ql, q_addr + QK_LO + kd * 32);
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        const uint32_t base = part * S_LO + kd * 16 * GC_LV * 2;
        uint32_t sb[4], s1[2];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          ldsm4_t(sb, s_addr + base + j * 32);
          mma16816(acc[2 * j], qh, sb[0], sb[1]);
          mma16816(acc[2 * j + 1], qh, sb[2], sb[3]);
          if (part == 0) {
            mma16816(acc[2 * j], ql, sb[0], sb[1]);
            mma16816(acc[2 * j + 1], ql, sb[2], sb[3]);
          }
        }
        ldsm2_t(s1, s1_addr + base);
        mma16816(acc[4], qh, s1[0], s1[1]);
        if (part == 0) mma16816(acc[4], ql, s1[0], s1[1]);
      }
#pragma unroll
      for (int kk = 0; kk < GC_L / 16; ++kk) {
        if (kk > rs) continue;
        const uint32_t at = k_addr + (uint32_t)(kk * 16 * (DKP + 8) * 2 + kd * 32);
        uint32_t kh[4], kl[4];
        ldsm4(kh, at);
        ldsm4(kl, at + QK_LO);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          mma16816(sc[kk][j], qh, kh[2 * j], kh[2 * j + 1]);
          mma16816(sc[kk][j], qh, kl[2 * j], kl[2 * j + 1]);
          mma16816(sc[kk][j], ql, kh[2 * j], kh[2 * j + 1]);
        }
      }
    }
    {
      const float g0 = S.carry[r0], g1 = S.carry[r0 + 8];
#pragma unroll
      for (int j = 0; j < 5; ++j) {
        acc[j][0] *= g0; acc[j][1] *= g0;
        acc[j][2] *= g1; acc[j][3] *= g1;
      }
    }
    const float A0 = S.A[r0], A1 = S.A[r0 + 8];
#pragma unroll
    for (int kk = 0; kk < GC_L / 16; ++kk) {
      if (kk > rs) continue;
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {                          // {rows, rows + 8} x {tokens 0-7, tokens 8-15}
        const int j = x >> 1, r = x & 1, key = kk * 16 + j * 8 + (lane & 3) * 2, t = r0 + r * 8;
        const float At = r ? A1 : A0;
        const float p0 = key <= t ? sc[kk][j][r * 2] * gc_ex2(At + S.B[key]) : 0.f;
        const float p1 = key + 1 <= t ? sc[kk][j][r * 2 + 1] * gc_ex2(At + S.B[key + 1]) : 0.f;
        split_bf16(p0, p1, ph[x], pl[x]);
      }
      const uint32_t base = (uint32_t)(kk * 16 * GC_LV * 2);
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        uint32_t vb[4];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          ldsm4_t(vb, v_addr + part * WV_LO + base + j * 32);
          mma16816(acc[2 * j], ph, vb[0], vb[1]);
          mma16816(acc[2 * j + 1], ph, vb[2], vb[3]);
          if (part == 0) {
            mma16816(acc[2 * j], pl, vb[0], vb[1]);
            mma16816(acc[2 * j + 1], pl, vb[2], vb[3]);
          }
        }
      }
      uint32_t v1[2];                                        // ones and zeros: no second part
      ldsm2_t(v1, v1_addr + base);
      mma16816(acc[4], ph, v1[0], v1[1]);
      mma16816(acc[4], pl, v1[0], v1[1]);
    }
    float sq[2] = {0.f, 0.f};
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const float nq = __shfl_sync(0xffffffffu, acc[4][2 * r], lane & ~3);
      const float unit = 1.0f / (fmaxf(fabsf(nq), S.low[r0 + r * 8]) + a.unit_eps);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[j][2 * r] *= unit;
        acc[j][2 * r + 1] *= unit;
        sq[r] = fmaf(acc[j][2 * r], acc[j][2 * r], fmaf(acc[j][2 * r + 1], acc[j][2 * r + 1], sq[r]));
      }
      sq[r] += __shfl_xor_sync(0xffffffffu, sq[r], 1);
      sq[r] += __shfl_xor_sync(0xffffffffu, sq[r], 2);
      if ((lane & 3) == 0) S.part[half][r0 + r * 8] = sq[r];
    }
    __syncthreads();                                         // everyone has read the state; the sums are there
    if (CS > 1) {
      if (tid < GC_L) S.ssq[ch & 1][tid] = S.part[0][tid] + S.part[1][tid];
      __syncwarp();
      asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    }
    // output gates on their way while the state advances
    float2 gate[4][2];
#pragma unroll
    for (int r = 0; r < 2; ++r)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = r0 + r * 8, c = half * 32 + j * 8 + (lane & 3) * 2;
        gate[j][r] = make_float2(0.f, 0.f);
        if (t < n && c < nv)
          gate[j][r] = *reinterpret_cast<const float2*>(a.proj + ((size_t)off + ch * GC_L + t) * a.ldp + a.g_off + h * V + c0 + c);
      }

    // ---- state
    const float decay = S.decay;
#pragma unroll
    for (int j = 0; j < NTW; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) st[j][e] *= decay;
#pragma unroll
    for (int kk = 0; kk < GC_L / 16; ++kk) {
      uint32_t kh[4], kl[4];
      ldsm4_t(kh, kt_addr + kk * 16 * (DKP + 8) * 2);
      ldsm4_t(kl, kt_addr + QK_LO + kk * 16 * (DKP + 8) * 2);
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        const uint32_t base = wv_addr + part * WV_LO + kk * 16 * GC_LV * 2;
#pragma unroll
        for (int j = 0; j < NTW; j += 2) {
          constexpr int LAST = NTW - 1;
          const int t = tile0 + j;
          if (t >= GC_NT) continue;
          if (j < LAST && t + 1 < GC_NT) {
            uint32_t b[4];
            ldsm4_t(b, base + t * 16 + (lane >> 4) * 16);
            const int j1 = j < LAST ? j + 1 : j;
            mma16816(st[j], kh, b[0], b[1]);
            mma16816(st[j1], kh, b[2], b[3]);
            if (part == 0) {
              mma16816(st[j], kl, b[0], b[1]);
              mma16816(st[j1], kl, b[2], b[3]);
            }
          } else {
            uint32_t b[2];
            ldsm2_t(b, base + t * 16);
            mma16816(st[j], kh, b[0], b[1]);
            if (part == 0) mma16816(st[j], kl, b[0], b[1]);
          }
        }
      }
    }
    if (ch + 1 < n_chunks) publish();

    // ---- outputs
    if (CS > 1) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = r0 + r * 8;
      float tot = 0.f;
      if (CS > 1) {
        const uint32_t at = smem_u32(&S.ssq[ch & 1][t]);
        for (int q = 0; q < CS; ++q) tot += ld_dsmem_f32(at, q);
      } else {
        tot = S.part[0][t] + S.part[1][t];
      }
      const float inv = 1.0f / sqrtf(tot / (float)V + a.eps);
      if (t >= n) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int c = half * 32 + j * 8 + (lane & 3) * 2;
        if (c >= nv) continue;
        const int col = h * V + c0 + c;
        const float2 w = *reinterpret_cast<const float2*>(a.onorm + col);
        *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(a.out) + ((size_t)off + ch * GC_L + t) * a.ldo + col) =
            pack_bf16(acc[j][2 * r] * inv * w.x * gc_sigmoid(gate[j][r].x), acc[j][2 * r + 1] * inv * w.y * gc_sigmoid(gate[j][r].y));
      }
    }
    __syncwarp();
  }
#pragma unroll
  for (int j = 0; j < NTW; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      bool real;
      const size_t at = state_at(j, e, real);
      if (real && (rank == 0 || (tile0 + j) * 8 < GC_EV)) M[at] = st[j][e];      // the normaliser once
    }
  if (rank == 0 && tid == 0) *top = m_run;
  __syncwarp();
  if (CS > 1) cluster_sync();                                // nobody leaves while its sums are read
}

template <int DKP>
static int gated_chunk_launch(const ScanArgs& a, cudaStream_t st) {
  const int cs = (a.V + GC_EV - 1) / GC_EV, bytes = (int)sizeof(GcShared<DKP>);
  CUDA_CHECK_RET(cudaFuncSetAttribute(gated_chunk_kernel<DKP>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
  return launch_cluster(gated_chunk_kernel<DKP>, dim3(a.H * cs, a.r.n_seq), dim3(GC_THREADS), bytes, st, a.pdl, cs, a, cs);
}

}  // namespace smc

// Whether the chunked form takes heads of D key rows and V value columns.
SMC_API int smc_gated_chunk_takes(int D, int V) { return D % 4 == 0 && D <= 128 && V % 4 == 0 && V <= 8 * smc::GC_EV; }

// The gated form in bf16, 64 tokens at a time; arguments as for smc_memory_scan.
SMC_API int smc_gated_chunk(const smc::ScanArgs* a, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_seq <= 0) return 0;
  if (!smc_gated_chunk_takes(a->D, a->V) || (a->ldp | a->r_off | a->k_off | a->v_off | a->g_off) % 4 || a->ldo % 2 || a->H < 1 ||
      a->r.n_seq > 65535)
    return -124;
  if (a->D <= 32) return gated_chunk_launch<32>(*a, st);
  if (a->D <= 64) return gated_chunk_launch<64>(*a, st);
  return gated_chunk_launch<128>(*a, st);
}
