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
constexpr int GC_THREADS = 512;
constexpr int GC_WARPS = GC_THREADS / 32;
constexpr int GC_MAX_CTAS = 8;                   // of a head

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
  __nv_bfloat16 p_room[DKP >= 64 ? 8 : 2 * GC_L * GC_LV];                // weights inside the chunk; they follow the queries into bq
  struct Gates { float A[GC_L], B[GC_L], carry[GC_L], low[GC_L], w[GC_L], decay, pad[3]; } gates[2];        // A, B in units of ln 2
  float nq[GC_L], part[4][GC_L], ssq[2][GC_L];
};

template <int DKP>
__global__ void __launch_bounds__(GC_THREADS, 1) gated_chunk_kernel(const ScanArgs a, int CS) {
  constexpr int KD = DKP / 16, GROUPS = GC_WARPS / KD, NTW = (GC_NT + GROUPS - 1) / GROUPS;
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

  // ---- fetching: a thread stays with its columns
  constexpr int QSTEP = GC_THREADS / (DKP / 4), VSTEP = GC_THREADS / (GC_EV / 4);
  const int qt = tid / (DKP / 4), qc = tid % (DKP / 4) * 4, vt = tid / (GC_EV / 4), vc = tid % (GC_EV / 4) * 4;
  const float* q_src = a.proj + ((size_t)off + qt) * a.ldp + h * D + qc;
  const float* v_src = a.proj + ((size_t)off + vt) * a.ldp + a.v_off + h * V + c0 + vc;
  const uint32_t q_dst = smem_u32(&S.q[qt][qc]), k_dst = smem_u32(&S.k[qt][qc]), v_dst = smem_u32(&S.v[vt][vc]);
  auto fetch = [&](int chunk) {
    const int n = min(GC_L, len - chunk * GC_L);
    const float* p = q_src + (size_t)chunk * GC_L * a.ldp;
#pragma unroll
    for (int i = 0; i < GC_L / QSTEP; ++i) {
      const bool real = qt + i * QSTEP < n && qc < D;
      const float* src = real ? p + (size_t)i * QSTEP * a.ldp : a.proj;
      cp_async16(q_dst + i * QSTEP * DKP * 4, src + (real ? a.r_off : 0), real);
      cp_async16(k_dst + i * QSTEP * DKP * 4, src + (real ? a.k_off : 0), real);
    }
    p = v_src + (size_t)chunk * GC_L * a.ldp;
#pragma unroll
    for (int i = 0; i < GC_L / VSTEP; ++i) {
      const bool real = vt + i * VSTEP < n && vc < nv;
      cp_async16(v_dst + i * VSTEP * GC_EV * 4, real ? p + (size_t)i * VSTEP * a.ldp : a.proj, real);
    }
    cp_async_commit();
  };
  fetch(0);

  // ---- gates: one warp, a chunk ahead; running sums and maxima are a scan over pairs (sum of f, maximum), two tokens per lane
  const bool gate_warp = warp == GC_WARPS - 1;
  float m_run = 0.f, gi[2], gf[2];                           // gi, gf: gate logits of the chunk after
  auto fetch_gates = [&](int chunk) {
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const float* p = a.proj + ((size_t)off + min(chunk * GC_L + 2 * lane + j, len - 1)) * a.ldp + a.a_off + h;
      gi[j] = p[0];
      gf[j] = p[H];
    }
  };
  auto gates = [&](int chunk) {
    typename GcShared<DKP>::Gates& G = S.gates[chunk & 1];
    const float cap = a.gate_cap, bias_i = a.a_bias[h], bias_f = a.a_bias[H + h];
    float li[2], lf[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const bool ok = chunk * GC_L + 2 * lane + j < len;
      li[j] = ok ? cap * tanhf((gi[j] + bias_i) / cap) : -INFINITY;
      lf[j] = ok ? log_sigmoid_f(cap * tanhf((gf[j] + bias_f) / cap)) : 0.f;
    }
    fetch_gates(chunk + 1);
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
      G.A[t] = A[j] * LOG2E;
      G.B[t] = B[j] * LOG2E;
      G.carry[t] = expf(A[j] + m_run);
      G.low[t] = expf(-mt[j]);
      G.w[t] = expf(B[j] + a_end);
    }
    if (lane == 0) G.decay = expf(a_end + m_run);
    m_run = m_end;
  };
  if (gate_warp) {
    m_run = *top;
    fetch_gates(0);
    gates(0);
  }

  // ---- state: this warp's 16 key rows, NTW column tiles
  const int strip = warp % KD, tile0 = (warp / KD) * NTW;
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

  // ---- read-out: this warp's 16 tokens and 16 columns, and one of: a 16 x 16 block of the weights on or below the diagonal (ten
  // warps), the normaliser's read-out for 16 tokens (four), the next chunk's gates (one)
  const int quarter = warp >> 2, rs = (warp + quarter) & 3;  // token strips of all lengths share a scheduler
  const int r0 = rs * 16 + (lane >> 2);                      // this thread's tokens: r0 and r0 + 8
  constexpr int BLOCKS = 10;
  const bool has_block = warp < BLOCKS, has_norm = warp >= BLOCKS && warp < BLOCKS + 4;
  const int rb = has_norm ? warp - BLOCKS : warp >= 6 ? 3 : warp >= 3 ? 2 : warp >= 1 ? 1 : 0, cb = warp - rb * (rb + 1) / 2;
  const int q_lane = (lane & 15) * (DKP + 8) + (lane >> 4) * 8;
  const uint32_t q_addr = smem_u32(&S.bq[0][rs * 16][0] + q_lane), qb_addr = smem_u32(&S.bq[0][rb * 16][0] + q_lane);
  const uint32_t k_addr = smem_u32(&S.bk[0][(has_block ? cb : 0) * 16 + (lane & 7) + ((lane >> 4) << 3)][((lane >> 3) & 1) * 8]);
  const uint32_t v_addr = smem_u32(&S.bv[0][lane & 15][quarter * 16 + (lane >> 4) * 8]), v1_addr = smem_u32(&S.bv[0][lane & 15][GC_EV]);
  const uint32_t s_addr = smem_u32(&S.s_hi[lane & 15][quarter * 16 + (lane >> 4) * 8]), s1_addr = smem_u32(&S.s_hi[lane & 15][GC_EV]);
  constexpr uint32_t S_LO = sizeof(S.s_hi), WV_LO = sizeof(S.wv_hi), QK_LO = sizeof(S.bq[0]), P_LO = GC_L * GC_LV * 2;
  __nv_bfloat16* P = DKP >= 64 ? &S.bq[0][0][0] : S.p_room;  // [hi, lo][token][token of the chunk], pitch GC_LV
  const uint32_t p_lane = (uint32_t)(((lane & 15) * GC_LV + (lane >> 4) * 8) * 2);
  const uint32_t p_addr = smem_u32(P) + rs * 16 * GC_LV * 2 + p_lane, pn_addr = smem_u32(P) + rb * 16 * GC_LV * 2 + p_lane;
  const uint32_t kt_addr = smem_u32(&S.bk[0][(lane & 7) + ((lane >> 4) & 1) * 8][strip * 16 + ((lane >> 3) & 1) * 8]);
  const uint32_t wv_addr = smem_u32(&S.wv_hi[lane & 15][0]);

  float2 onorm[2];
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int c = quarter * 16 + j * 8 + (lane & 3) * 2;
    onorm[j] = c < nv ? *reinterpret_cast<const float2*>(a.onorm + h * V + c0 + c) : make_float2(0.f, 0.f);
  }

  for (int ch = 0; ch < n_chunks; ++ch) {
    const int n = min(GC_L, len - ch * GC_L);
    const typename GcShared<DKP>::Gates& G = S.gates[ch & 1];
    cp_async_wait<0>();
    __syncthreads();
    // ---- operands
#pragma unroll
    for (int i = 0; i < GC_L / QSTEP; ++i) {
      const int t = qt + i * QSTEP;
      const float4 q = load4((const float*)&S.q[t][qc]), k = load4((const float*)&S.k[t][qc]);
      uint2 hi, lo;
      split_bf16(q.x * a.r_scale, q.y * a.r_scale, hi.x, lo.x);
      split_bf16(q.z * a.r_scale, q.w * a.r_scale, hi.y, lo.y);
      *reinterpret_cast<uint2*>(&S.bq[0][t][qc]) = hi;
      *reinterpret_cast<uint2*>(&S.bq[1][t][qc]) = lo;
      split_bf16(k.x, k.y, hi.x, lo.x);
      split_bf16(k.z, k.w, hi.y, lo.y);
      *reinterpret_cast<uint2*>(&S.bk[0][t][qc]) = hi;
      *reinterpret_cast<uint2*>(&S.bk[1][t][qc]) = lo;
    }
    auto values = [&](int t, int c, float4 v) {
      const float w = G.w[t];
      uint2 hi, lo;
      split_bf16(v.x, v.y, hi.x, lo.x);
      split_bf16(v.z, v.w, hi.y, lo.y);
      *reinterpret_cast<uint2*>(&S.bv[0][t][c]) = hi;
      *reinterpret_cast<uint2*>(&S.bv[1][t][c]) = lo;
      split_bf16(w * v.x, w * v.y, hi.x, lo.x);
      split_bf16(w * v.z, w * v.w, hi.y, lo.y);
      *reinterpret_cast<uint2*>(&S.wv_hi[t][c]) = hi;
      *reinterpret_cast<uint2*>(&S.wv_lo[t][c]) = lo;
    };
#pragma unroll
    for (int i = 0; i < GC_L / VSTEP; ++i) values(vt + i * VSTEP, vc, load4((const float*)&S.v[vt + i * VSTEP][vc]));
    if (tid < GC_L * 2) {                                    // the normaliser's columns
      const int t = tid >> 1;
      values(t, GC_EV + (tid & 1) * 4, make_float4((tid & 1) == 0 && t < n ? 1.f : 0.f, 0.f, 0.f, 0.f));
    }
    __syncthreads();
    if (ch + 1 < n_chunks) fetch(ch + 1);

    // ---- products with the state, weights
    float acc[2][4], ex[2][4];                               // read-out; block of weights or the normaliser's read-out
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[j][e] = ex[j][e] = 0.f;
#pragma unroll
    for (int kd = 0; kd < KD; ++kd) {
      uint32_t qh[4], ql[4], sb[4];
      ldsm4(qh, q_addr + kd * 32);
      ldsm4(ql, q_addr + QK_LO + kd * 32);
      const uint32_t at = s_addr + kd * 16 * GC_LV * 2;
      ldsm4_t(sb, at);
      mma16816(acc[0], qh, sb[0], sb[1]);
      mma16816(acc[1], qh, sb[2], sb[3]);
      mma16816(acc[0], ql, sb[0], sb[1]);
      mma16816(acc[1], ql, sb[2], sb[3]);
      ldsm4_t(sb, at + S_LO);
      mma16816(acc[0], qh, sb[0], sb[1]);
      mma16816(acc[1], qh, sb[2], sb[3]);
    }
    uint32_t ph[4], pl[4];
    if (has_block) {
#pragma unroll
      for (int kd = 0; kd < KD; ++kd) {
        uint32_t qh[4], ql[4], kh[4], kl[4];
        ldsm4(qh, qb_addr + kd * 32);
        ldsm4(kh, k_addr + kd * 32);
        ldsm4(ql, qb_addr + QK_LO + kd * 32);
        ldsm4(kl, k_addr + QK_LO + kd * 32);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          mma16816(ex[j], qh, kh[2 * j], kh[2 * j + 1]);
          mma16816(ex[j], qh, kl[2 * j], kl[2 * j + 1]);
          mma16816(ex[j], ql, kh[2 * j], kh[2 * j + 1]);
        }
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) {                          // {rows, rows + 8} x {tokens 0-7, tokens 8-15}
        const int j = x >> 1, r = x & 1, key = cb * 16 + j * 8 + (lane & 3) * 2, t = rb * 16 + (lane >> 2) + r * 8;
        const float At = G.A[t];
        const float p0 = key <= t ? ex[j][r * 2] * gc_ex2(At + G.B[key]) : 0.f;
        const float p1 = key + 1 <= t ? ex[j][r * 2 + 1] * gc_ex2(At + G.B[key + 1]) : 0.f;
        split_bf16(p0, p1, ph[x], pl[x]);
      }
    } else if (has_norm) {
#pragma unroll
      for (int kd = 0; kd < KD; ++kd) {
        uint32_t qh[4], ql[4], s1[2];
        ldsm4(qh, qb_addr + kd * 32);
        ldsm4(ql, qb_addr + QK_LO + kd * 32);
        ldsm2_t(s1, s1_addr + kd * 16 * GC_LV * 2);
        mma16816(ex[0], qh, s1[0], s1[1]);
        mma16816(ex[0], ql, s1[0], s1[1]);
        ldsm2_t(s1, s1_addr + S_LO + kd * 16 * GC_LV * 2);
        mma16816(ex[0], qh, s1[0], s1[1]);
      }
      const float g0 = G.carry[rb * 16 + (lane >> 2)], g1 = G.carry[rb * 16 + (lane >> 2) + 8];
      ex[0][0] *= g0;
      ex[0][2] *= g1;
    } else if (gate_warp && ch + 1 < n_chunks) {
      gates(ch + 1);
    }
    {
      const float g0 = G.carry[r0], g1 = G.carry[r0 + 8];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        acc[j][0] *= g0; acc[j][1] *= g0;
        acc[j][2] *= g1; acc[j][3] *= g1;
      }
    }
    __syncthreads();                                         // the queries have been read
    if (has_block) {
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int at = (rb * 16 + (lane >> 2) + (x & 1) * 8) * GC_LV + cb * 16 + (x >> 1) * 8 + (lane & 3) * 2;
        *reinterpret_cast<uint32_t*>(P + at) = ph[x];
        *reinterpret_cast<uint32_t*>(P + GC_L * GC_LV + at) = pl[x];
      }
    }
    __syncthreads();
    // ---- products with the values
#pragma unroll
    for (int kk = 0; kk < GC_L / 16; ++kk) {
      if (kk > rs) continue;
      const uint32_t base = (uint32_t)(kk * 16 * GC_LV * 2);
      uint32_t vb[4];
      ldsm4(ph, p_addr + kk * 32);
      ldsm4(pl, p_addr + P_LO + kk * 32);
      ldsm4_t(vb, v_addr + base);
      mma16816(acc[0], ph, vb[0], vb[1]);
      mma16816(acc[1], ph, vb[2], vb[3]);
      mma16816(acc[0], pl, vb[0], vb[1]);
      mma16816(acc[1], pl, vb[2], vb[3]);
      ldsm4_t(vb, v_addr + WV_LO + base);
      mma16816(acc[0], ph, vb[0], vb[1]);
      mma16816(acc[1], ph, vb[2], vb[3]);
    }
    if (has_norm) {                                          // ones and zeros: no second part
      for (int kk = 0; kk <= rb; ++kk) {
        uint32_t v1[2];
        ldsm4(ph, pn_addr + kk * 32);
        ldsm4(pl, pn_addr + P_LO + kk * 32);
        ldsm2_t(v1, v1_addr + kk * 16 * GC_LV * 2);
        mma16816(ex[0], ph, v1[0], v1[1]);
        mma16816(ex[0], pl, v1[0], v1[1]);
      }
      if ((lane & 3) == 0) {
        S.nq[rb * 16 + (lane >> 2)] = ex[0][0];
        S.nq[rb * 16 + (lane >> 2) + 8] = ex[0][2];
      }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float sq = 0.f;
#pragma unroll
      for (int j = 0; j < 2; ++j) sq = fmaf(acc[j][2 * r], acc[j][2 * r], fmaf(acc[j][2 * r + 1], acc[j][2 * r + 1], sq));
      sq += __shfl_xor_sync(0xffffffffu, sq, 1);
      sq += __shfl_xor_sync(0xffffffffu, sq, 2);
      if ((lane & 3) == 0) S.part[quarter][r0 + r * 8] = sq;
    }
    __syncthreads();                                         // everyone has read the state; the sums are there
    if (CS > 1) {
      if (tid < GC_L) S.ssq[ch & 1][tid] = (S.part[0][tid] + S.part[1][tid]) + (S.part[2][tid] + S.part[3][tid]);
      __syncwarp();
      asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    }
    // output gates on their way while the state advances
    float2 gate[2][2];
#pragma unroll
    for (int r = 0; r < 2; ++r)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = r0 + r * 8, c = quarter * 16 + j * 8 + (lane & 3) * 2;
        gate[j][r] = make_float2(0.f, 0.f);
        if (t < n && c < nv)
          gate[j][r] = *reinterpret_cast<const float2*>(a.proj + ((size_t)off + ch * GC_L + t) * a.ldp + a.g_off + h * V + c0 + c);
      }

    // ---- state
    const float decay = G.decay;
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
    float tot[2] = {0.f, 0.f};
    if (CS > 1) {
      asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
      const uint32_t at = smem_u32(&S.ssq[ch & 1][r0]);
#pragma unroll
      for (int q = 0; q < GC_MAX_CTAS; ++q)
        if (q < CS) {
          const uint32_t there = dsmem_map(at, (uint32_t)q);
          tot[0] += ld_dsmem_f32_at(there);
          tot[1] += ld_dsmem_f32_at(there + 32u);
        }
    } else {
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = r0 + r * 8;
        tot[r] = (S.part[0][t] + S.part[1][t]) + (S.part[2][t] + S.part[3][t]);
      }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = r0 + r * 8;
      const float unit = 1.0f / (fmaxf(fabsf(S.nq[t]), G.low[t]) + a.unit_eps), inv = unit / sqrtf(tot[r] * unit * unit / (float)V + a.eps);
      if (t >= n) continue;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int c = quarter * 16 + j * 8 + (lane & 3) * 2;
        if (c >= nv) continue;
        *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(a.out) + ((size_t)off + ch * GC_L + t) * a.ldo + h * V + c0 + c) =
            pack_bf16(acc[j][2 * r] * inv * onorm[j].x * gc_sigmoid(gate[j][r].x), acc[j][2 * r + 1] * inv * onorm[j].y * gc_sigmoid(gate[j][r].y));
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
  if (rank == 0 && gate_warp && lane == 0) *top = m_run;
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
SMC_API int smc_gated_chunk_takes(int D, int V) { return D % 4 == 0 && D <= 128 && V % 4 == 0 && V <= smc::GC_MAX_CTAS * smc::GC_EV; }

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
