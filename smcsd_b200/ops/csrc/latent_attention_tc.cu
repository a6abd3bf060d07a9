// Latent attention on the 5th-generation tensor cores (tcgen05 + tensor memory).
//
// All heads of a token attend to the same cached rows of R values (R padded to panels of 64), so the query rows of a block
// of tokens - row = token * heads + head, up to 128 per CTA - form one M = 128 operand, and a tile of 64 cached rows serves
// as keys and as values from the same shared-memory bytes:
//     S = Q C^T        UMMA 128 x 64 x R, C taken K-major
//     softmax          two threads per query row (both take the row's maximum, each exponentiates half of the tile's
//                      columns), causal and window limit per row, an optional sink logit per head in the sum, P as bf16 into a SWIZZLE_128B tile
//     O += P C         UMMA 128 x R x 64 accumulating in tensor memory, C taken MN-major
// Two score buffers (64 columns each) and up to 384 output columns live in tensor memory; wider latents split their output
// columns over two CTAs that both compute the scores.  The exponent reference of a row only moves when its maximum grew by
// more than 2^8; only then is its part of O rescaled in tensor memory.
// Cached rows live one page per token: a tile of 64 consecutive pages is fetched with one TMA box per panel, a scattered one
// is gathered by four loader warps with 16-byte cp.async copies into the same swizzled layout (TMA gathers of four rows each
// measured 1.5 times slower); the copies arrive on the tile's mbarrier by themselves, so loaders never wait for one to land.  Key ranges may be split over
// the CTAs of a thread-block cluster (few sequences, long contexts): every split parks its unnormalised rows in its own shared
// memory and the CTAs merge them through distributed shared memory, each a share of the rows.
// The work list (ragged.cuh) mixes prompts, portions of prompts and single tokens; query rows never mix sequences.
// Every mbarrier wait is bounded; a timeout raises a status bit and every role unwinds.
#include "latent_attention.cuh"
#include "tmap_host.h"

namespace smc {

constexpr int LT_BK = 64;                       // cached rows per tile
constexpr int LT_LOADERS = 4;
constexpr int LT_THREADS = (9 + LT_LOADERS) * 32;   // warps 0..7 softmax (4..7: the upper half of the columns), 8 MMA, 9.. loaders
constexpr int LT_PANEL_Q = 128 * 128;           // bytes of one [128 rows][64 values] panel
constexpr int LT_PANEL_C = LT_BK * 128;
constexpr int LT_O_COL = 2 * LT_BK;             // first output column in tensor memory
constexpr int LT_MAX_STAGES = 6;
constexpr int LT_MAX_SPLITS = 8;                // CTAs of a cluster
constexpr float LT_LOG2E = 1.4426950408889634f;

// NPAN: panels of 64 values per cached row.  Ring depth within 227 KB next to the Q tile and two P tiles.
template <int NPAN> struct LtCfg {
  static constexpr int VSPLIT = NPAN > 6 ? 2 : 1;                    // CTAs sharing the output columns
  static constexpr int OPAN = (NPAN + VSPLIT - 1) / VSPLIT;          // output panels per CTA (the second may have fewer)
  static constexpr int FIXED = NPAN * LT_PANEL_Q + 2 * LT_PANEL_Q;
  static constexpr int FIT = (231000 - 1024 - FIXED) / (NPAN * LT_PANEL_C);
  static constexpr int STAGES = FIT > LT_MAX_STAGES ? LT_MAX_STAGES : FIT;
  static constexpr int SMEM = FIXED + STAGES * NPAN * LT_PANEL_C + 1024;
  static constexpr int OLD = OPAN * 64 + 1;                          // row pitch of the parked rows (floats)
  static constexpr int STATS = FIXED + STAGES * NPAN * LT_PANEL_C - 2048;   // row statistics, at the end of the P buffers
  static constexpr int TMEM_COLS = OPAN <= 2 ? 256 : 512;
  static_assert(STAGES >= 1 && 128 * OLD * 4 <= STATS, "a tile and the parked rows must fit");
};

struct LatentTcParams {
  const __nv_bfloat16* pool;     // [pages + 1, ldc]
  __nv_bfloat16* out;            // [T * H, ldc]
  const int* block_table;
  int bt_stride, bt_rows, n_pages, H, ldc, KS, MT, T;
  float scale_log2;
  int window;                    // 0: all
  const float* sink;             // [H] (null: none)
  Ragged r;
  int* status;
  int pdl;
};

struct LtShared {
  uint64_t q_full, c_full[LT_MAX_STAGES], c_empty[LT_MAX_STAGES], s_full[2], s_empty[2], p_full[2], p_empty[2];
  uint32_t tmem_slot;
  volatile int abort;
};

__device__ __forceinline__ bool lt_wait(LtShared& S, int* status, uint64_t* bar, uint32_t parity) {
  if (mbar_try_wait(bar, parity)) return true;
  if (S.abort) return false;
  const long long t0 = clock64();
  for (;;) {
    for (int i = 0; i < 64; ++i)
      if (mbar_try_wait(bar, parity)) return true;
    if (S.abort) return false;
    if (clock64() - t0 > SMC_SPIN_CYCLES) {
      atomicOr(status, SMC_ERR_BARRIER_TIMEOUT);
      S.abort = 1;
      return false;
    }
  }
}

__device__ __forceinline__ float lt_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t lt_pack(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}

template <int NPAN>
__global__ void __launch_bounds__(LT_THREADS, 1) latent_tc_kernel(const LatentTcParams p, const __grid_constant__ CUtensorMap tmC,
                                                                  const __grid_constant__ CUtensorMap tmQ) {
  using C = LtCfg<NPAN>;
  constexpr int STAGES = C::STAGES, CPR = NPAN * 8, KPW = LT_BK / LT_LOADERS, C_BYTES = NPAN * LT_PANEL_C;
  extern __shared__ uint8_t lt_raw[];
  __shared__ LtShared S;
  const uint32_t raw = smem_u32(lt_raw);
  uint8_t* q_s = lt_raw + (((raw + 1023u) & ~1023u) - raw);
  uint8_t* c_s = q_s + NPAN * LT_PANEL_Q;
  uint8_t* p_s = c_s + STAGES * C_BYTES;
  float* st_m = reinterpret_cast<float*>(q_s + C::STATS);   // [128] reference exponents (log2 units), [128] sums of a key split,
  float* st_l = st_m + 128;                                 // [2][128] sums of the two halves of the columns; P is idle by then
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    mbar_init(&S.q_full, 1);
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&S.c_full[s], LT_LOADERS * 32);
      mbar_init(&S.c_empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&S.s_full[i], 1);
      mbar_init(&S.s_empty[i], 8);
      mbar_init(&S.p_full[i], 8);
      mbar_init(&S.p_empty[i], 1);
    }
    S.abort = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmC);
    tma_prefetch_desc(&tmQ);
  }
  if (warp == 8) {
    tmem_alloc(&S.tmem_slot, C::TMEM_COLS);
    tmem_relinquish();
  }
  if (p.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }

  // ---- this CTA's rows and keys --------------------------------------------------------------------------------------
  const int vs = blockIdx.x % C::VSPLIT, mt = (blockIdx.x / C::VSPLIT) % p.MT, blk = blockIdx.x / (C::VSPLIT * p.MT), ks = blockIdx.y;
  RaggedBlock b = ragged_block(p.r, blk);
  if (b.row < 0 || b.row >= p.bt_rows || b.prefix < 0 || b.prefix + b.len > p.bt_stride || b.off < 0 || b.off + b.len > p.T) {
    if (threadIdx.x == 0) atomicOr(p.status, SMC_ERR_BOUNDS);
    b.n = 0;
    b.row = 0;
  }
  const int row0 = mt * 128, n_rows = min(128, max(0, b.n) * p.H - row0);      // <= 0: nothing to do
  const int g_row0 = (b.off + b.start) * p.H + row0;                           // in the [T * H] query rows
  const int pos0 = b.prefix + b.start;                                         // position of the block's first token
  const int lim_min = pos0 + row0 / p.H + 1;                                   // keys the tile's first row sees
  const int n_keys = n_rows > 0 ? pos0 + (row0 + n_rows - 1) / p.H + 1 : 0;
  const int lo_min = p.window > 0 ? max(0, lim_min - p.window) : 0;            // first key the tile's first row sees
  const int lo_max = p.window > 0 ? max(0, n_keys - p.window) : 0;             // .. the last row
  int per = (n_keys - lo_min + p.KS - 1) / p.KS;
  per = (per + LT_BK - 1) / LT_BK * LT_BK;
  const int kb = lo_min + ks * per, ke = min(n_keys, kb + per);
  const int n_tiles = ke > kb ? (ke - kb + LT_BK - 1) / LT_BK : 0;
  const int vpan = vs * C::OPAN, n_opan = min(C::OPAN, NPAN - vpan);           // this CTA's output panels

  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = S.tmem_slot;
  const uint32_t tO = tmem_base + LT_O_COL;

  if (warp >= 9) {
    // ================================================================= loaders
    const int lw = warp - 9;
    const uint64_t pol = l2_policy_evict_last();      // other row tiles and splits read the same rows
    if (lw == 0 && lane == 0 && n_tiles > 0) {
      // whole boxes of 128 rows: what the rows behind the queries contain only reaches their own outputs
      mbar_expect_tx(&S.q_full, NPAN * LT_PANEL_Q);
      for (int pan = 0; pan < NPAN; ++pan) tma_load_2d(q_s + pan * LT_PANEL_Q, &tmQ, &S.q_full, pan * 64, g_row0, pol);
    }
    const int* bt = p.block_table + (size_t)b.row * p.bt_stride;
    // every loader warp reads all 64 page ids of a tile (lane l: keys l and l + 32), so all take the same path
    auto page_of = [&](int tile, int half) {
      const int key = kb + tile * LT_BK + half * 32 + lane;
      return tile < n_tiles && key < ke ? bt[key] : 0;
    };
    auto checked = [&](int page) {                    // at the point of use: a check at the load would wait for it
      if (page < 0 || page > p.n_pages) { atomicOr(p.status, SMC_ERR_BOUNDS); page = 0; }
      return page;
    };
    constexpr int PD = 4;                             // page ids are fetched this many tiles ahead
    int issued = 0, pg[PD][2];
#pragma unroll
    for (int u = 0; u < PD; ++u) {
      pg[u][0] = page_of(u, 0);
      pg[u][1] = page_of(u, 1);
    }
    bool go = true;
    for (int j0 = 0; go && j0 < n_tiles; j0 += PD) {
#pragma unroll
      for (int u = 0; u < PD; ++u) {
        const int j = j0 + u;
        if (j >= n_tiles) break;
        const int st = j % STAGES, use = j / STAGES;
        const bool ok = use < 1 || lt_wait(S, p.status, &S.c_empty[st], (uint32_t)(use - 1) & 1u);
        if (!__all_sync(0xffffffffu, ok)) { go = false; break; }
        const int pa = checked(pg[u][0]), pb = checked(pg[u][1]);
        pg[u][0] = page_of(j + PD, 0);
        pg[u][1] = page_of(j + PD, 1);
        const int base = __shfl_sync(0xffffffffu, pa, 0), key_end = kb + (j + 1) * LT_BK;
        const bool asc = __all_sync(0xffffffffu, pa == base + lane && pb == base + 32 + lane);
        // descending pages reverse the keys inside the tile, which is fine where every row sees all of them
        const bool desc = __all_sync(0xffffffffu, pa == base - lane && pb == base - 32 - lane) && base >= LT_BK && key_end <= lim_min &&
                          key_end - LT_BK >= lo_max;
        const bool run = key_end <= ke && base >= 1 && (asc || desc);
        uint8_t* c_ptr = c_s + (size_t)st * C_BYTES;
        if (run) {
          if (lw == 0 && lane == 0) {
            mbar_expect_tx(&S.c_full[st], C_BYTES);
            for (int pan = 0; pan < NPAN; ++pan)
              tma_load_2d(c_ptr + pan * LT_PANEL_C, &tmC, &S.c_full[st], pan * 64, asc ? base : base - (LT_BK - 1), pol);
          } else {
            mbar_arrive(&S.c_full[st]);
          }
        } else {
          const uint32_t c_t = smem_u32(c_ptr);
          const int mine = lw < 2 ? pa : pb;          // this warp's 16 keys sit in lanes (lw & 1) * 16 ..
#pragma unroll
          for (int i = 0; i < KPW * CPR / 32; ++i) {
            const int idx = i * 32 + lane, kl = idx / CPR, c = idx % CPR, key = lw * KPW + kl;
            const int pgi = __shfl_sync(0xffffffffu, mine, (lw & 1) * 16 + kl);
            const uint32_t dst = c_t + (uint32_t)((c >> 3) * LT_PANEL_C + key * 128 + (((c & 7) ^ (key & 7)) << 4));
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(p.pool + (size_t)pgi * p.ldc + c * 8) : "memory");
          }
          // this thread's arrival follows its copies
          asm volatile("cp.async.mbarrier.arrive.noinc.shared::cta.b64 [%0];" ::"r"(smem_u32(&S.c_full[st])) : "memory");
        }
        ++issued;
      }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    // TMA copies still in flight after an abort must land before the CTA ends
    __syncwarp();
    if (S.abort && lw == 0 && lane == 0) {
      if (n_tiles > 0) (void)mbar_wait(&S.q_full, 0);
      for (int t = max(0, issued - STAGES); t < issued; ++t) (void)mbar_wait(&S.c_full[t % STAGES], (uint32_t)(t / STAGES) & 1u);
    }
  } else if (warp == 8) {
    // ================================================================= MMA issuer (one thread)
    if (elect_one()) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(128, LT_BK);
      const uint32_t q_addr = smem_u32(q_s), p_addr = smem_u32(p_s), c_addr0 = smem_u32(c_s);
      auto issue_s = [&](int j) -> bool {
        const int st = j % STAGES;
        if (!lt_wait(S, p.status, &S.c_full[st], (uint32_t)(j / STAGES) & 1u)) return false;
        if (j >= 2 && !lt_wait(S, p.status, &S.s_empty[j & 1], (uint32_t)((j >> 1) - 1) & 1u)) return false;
        fence_proxy_async();                          // gathered rows were written through the generic proxy
        tc_fence_after();
        const uint32_t c_addr = c_addr0 + (uint32_t)st * C_BYTES;
#pragma unroll
        for (int pan = 0; pan < NPAN; ++pan)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_ss(tmem_base + (uint32_t)(j & 1) * LT_BK, umma_desc_k_sw128(q_addr + pan * LT_PANEL_Q) + 2 * k,
                         umma_desc_k_sw128(c_addr + pan * LT_PANEL_C) + 2 * k, idesc_s, (pan | k) ? 1u : 0u);
        umma_commit(&S.s_full[j & 1]);
        return true;
      };
      bool ok = n_tiles > 0 && lt_wait(S, p.status, &S.q_full, 0) && issue_s(0);
      for (int j = 0; ok && j < n_tiles; ++j) {
        if (STAGES > 1 && j + 1 < n_tiles && !issue_s(j + 1)) break;     // next tile's scores overlap this tile's softmax
        if (!lt_wait(S, p.status, &S.p_full[j & 1], (uint32_t)(j >> 1) & 1u)) break;
        tc_fence_after();
        const int st = j % STAGES;
        const uint32_t pj = p_addr + (uint32_t)(j & 1) * LT_PANEL_Q;
        const uint32_t v_addr = c_addr0 + (uint32_t)st * C_BYTES + (uint32_t)vpan * LT_PANEL_C;
        for (int g = 0; g < n_opan; g += 4) {                            // at most 256 output columns per instruction
          const uint32_t idesc_o = umma_idesc_bf16(128, min(4, n_opan - g) * 64) | (1u << 16);   // B operand is MN-major
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_ss(tO + (uint32_t)g * 64u, umma_desc_k_sw128(pj) + 2 * k,
                         umma_desc_mn_sw128(v_addr + g * LT_PANEL_C + k * 2048, LT_PANEL_C), idesc_o, (j | k) ? 1u : 0u);
        }
        umma_commit(&S.c_empty[st]);
        umma_commit(&S.p_empty[j & 1]);                                  // also: O holds the sum over tiles 0..j
        if (STAGES == 1 && j + 1 < n_tiles && !issue_s(j + 1)) break;
      }
    }
    __syncwarp();
  } else {
    // ================================================================= softmax (two threads per query row)
    constexpr int HB = LT_BK / 2;                                        // columns this thread exponentiates
    const int half = warp >> 2, r = (warp & 3) * 32 + lane;
    const uint32_t lane_off = ((uint32_t)((warp & 3) * 32)) << 16;
    const bool real = r < n_rows;
    const int lim = real ? pos0 + (row0 + r) / p.H + 1 : ke;             // keys [0, lim) are visible (spare rows: unmasked)
    const int lo = real && p.window > 0 ? max(0, lim - p.window) : 0;    // .. from here on
    float m_ref = -INFINITY, l = 0.f;                                    // exponent reference (log2 domain), running sum
    bool alive = true;
    const bool idle = (warp & 3) * 32 >= n_rows;                         // no real row in this warp: keep the protocol only
    for (int j = 0; j < n_tiles; ++j) {
      const int nv = min(lim, ke) - kb - j * LT_BK;                      // columns [nl, nv) of this tile are visible (may be none)
      const int nl = lo - kb - j * LT_BK;
      if (!__all_sync(0xffffffffu, lt_wait(S, p.status, &S.s_full[j & 1], (uint32_t)(j >> 1) & 1u))) { alive = false; break; }
      tc_fence_after();
      uint32_t x[HB];
      float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      const bool full = __all_sync(0xffffffffu, nv >= LT_BK && nl <= 0);
      if (!idle) {
        const uint32_t ts = tmem_base + (uint32_t)(j & 1) * LT_BK + lane_off;
        uint32_t y[HB];                               // the other half: only its maximum is needed here
#pragma unroll
        for (int c0 = 0; c0 < HB; c0 += 16) {
          tmem_ld_32x32b_x16(ts + half * HB + c0, *reinterpret_cast<uint32_t(*)[16]>(&x[c0]));
          tmem_ld_32x32b_x16(ts + (half ^ 1) * HB + c0, *reinterpret_cast<uint32_t(*)[16]>(&y[c0]));
        }
        tmem_ld_wait();
        if (full) {
#pragma unroll
          for (int i = 0; i < HB; ++i) m4[i & 3] = fmaxf(m4[i & 3], fmaxf(__uint_as_float(x[i]), __uint_as_float(y[i])));
        } else {
          const int nx = nv - half * HB, ny = nv - (half ^ 1) * HB, lx = nl - half * HB, ly = nl - (half ^ 1) * HB;
#pragma unroll
          for (int i = 0; i < HB; ++i) {
            if (i < nx && i >= lx) m4[i & 3] = fmaxf(m4[i & 3], __uint_as_float(x[i]));
            if (i < ny && i >= ly) m4[i & 3] = fmaxf(m4[i & 3], __uint_as_float(y[i]));
          }
        }
      }
      tc_fence_before();                              // the scores are in registers: the buffer can take tile j + 2
      __syncwarp();
      if (lane == 0) mbar_arrive(&S.s_empty[j & 1]);
      const float mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3])) * p.scale_log2;
      const bool grow = mx > m_ref + 8.f;             // also true on the row's first visible key (m_ref = -inf)
      if (j >= 1 && __any_sync(0xffffffffu, grow)) {
        // PV of tile j - 1 must have completed before O is rescaled in tensor memory
        if (!__all_sync(0xffffffffu, lt_wait(S, p.status, &S.p_empty[(j - 1) & 1], (uint32_t)((j - 1) >> 1) & 1u))) { alive = false; break; }
        tc_fence_after();
        const float alpha = grow ? exp2f(m_ref - mx) : 1.f;
        for (int c0 = half * 32; c0 < n_opan * 64; c0 += (c0 & 16) ? 48 : 16) {     // this half's 32 columns of every panel
          uint32_t o[16];
          tmem_ld_32x32b_x16(tO + lane_off + c0, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
          tmem_st_32x32b_x16(tO + lane_off + c0, o);
        }
        tmem_st_wait();
        l *= alpha;
      }
      if (grow) m_ref = mx;
      // P buffer j & 1 was last read by PV of tile j - 2
      if (!__all_sync(0xffffffffu, j < 2 || lt_wait(S, p.status, &S.p_empty[j & 1], (uint32_t)((j - 2) >> 1) & 1u))) { alive = false; break; }
      uint8_t* prow = p_s + (j & 1) * LT_PANEL_Q + r * 128;
      if (idle) {
        if (j < 2) {                                  // rows without a query stay zero in both buffers
#pragma unroll
          for (int c = 0; c < 4; ++c) *reinterpret_cast<uint4*>(prow + ((half * 4 + c) << 4)) = make_uint4(0u, 0u, 0u, 0u);
        }
      } else {
        const float ref = m_ref == -INFINITY ? 0.f : m_ref;
        if (!full) {                                  // keys the row does not see: exp2 of -inf
          const int nx = nv - half * HB, lx = nl - half * HB;
#pragma unroll
          for (int i = 0; i < HB; ++i) x[i] = i < nx && i >= lx ? x[i] : 0xff800000u;
        }
        float s4[4] = {0.f, 0.f, 0.f, 0.f};
        uint32_t w[HB / 2];
#pragma unroll
        for (int i = 0; i < HB / 2; ++i) {
          w[i] = lt_pack(lt_ex2(fmaf(__uint_as_float(x[2 * i]), p.scale_log2, -ref)),
                         lt_ex2(fmaf(__uint_as_float(x[2 * i + 1]), p.scale_log2, -ref)));
          // the sum is taken over the rounded weights: they add up to one, and a lone heavy key carries no rounding error
          s4[(2 * i) & 3] += __uint_as_float(w[i] << 16);
          s4[(2 * i + 1) & 3] += __uint_as_float(w[i] & 0xffff0000u);
        }
#pragma unroll
        for (int c = 0; c < HB / 8; ++c) {            // 16-byte chunks of this row's 128 bytes
          const int cc = half * (HB / 8) + c;
          *reinterpret_cast<uint4*>(prow + ((cc ^ (r & 7)) << 4)) = make_uint4(w[c * 4], w[c * 4 + 1], w[c * 4 + 2], w[c * 4 + 3]);
        }
        l += (s4[0] + s4[1]) + (s4[2] + s4[3]);
      }
      tc_fence_before();
      fence_proxy_async();                            // P must be visible to the tensor core
      __syncwarp();
      if (lane == 0) mbar_arrive(&S.p_full[j & 1]);
    }
    // the last PV has completed when its P buffer is released: read O once
    if (alive && n_tiles > 0)
      alive = __all_sync(0xffffffffu, lt_wait(S, p.status, &S.p_empty[(n_tiles - 1) & 1], (uint32_t)((n_tiles - 1) >> 1) & 1u));
    tc_fence_after();
    const bool write = real && alive && !S.abort;
    st_l[128 + half * 128 + r] = l;
    asm volatile("bar.sync 1, 256;" ::: "memory");    // the eight softmax warps
    l = st_l[128 + r] + st_l[256 + r];
    if (p.KS > 1 && half == 0) {
      st_m[r] = write ? m_ref : -INFINITY;
      st_l[r] = write ? l : 0.f;                       // 0: this split holds nothing for the row
    }
    if (p.KS == 1 && p.sink != nullptr && write) l += exp2f(p.sink[(row0 + r) % p.H] * LT_LOG2E - m_ref);
    if (n_tiles > 0 && alive && !idle) {
      const float inv = l > 0.f ? 1.0f / l : 0.f;
      float* po = reinterpret_cast<float*>(q_s) + r * C::OLD;       // operands and tiles are no longer needed
      __nv_bfloat16* oo = p.out + ((size_t)g_row0 + r) * p.ldc + vpan * 64;
      for (int c0 = half * 32; c0 < n_opan * 64; c0 += (c0 & 16) ? 48 : 16) {
        uint32_t o[16];
        tmem_ld_32x32b_x16(tO + lane_off + c0, o);
        tmem_ld_wait();
        if (p.KS > 1) {
#pragma unroll
          for (int i = 0; i < 16; ++i) po[c0 + i] = __uint_as_float(o[i]);
        } else if (write) {
          uint32_t pk[8];
#pragma unroll
          for (int i = 0; i < 16; i += 2) pk[i >> 1] = lt_pack(__uint_as_float(o[i]) * inv, __uint_as_float(o[i + 1]) * inv);
          *reinterpret_cast<uint4*>(oo + c0) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
          *reinterpret_cast<uint4*>(oo + c0 + 8) = make_uint4(pk[4], pk[5], pk[6], pk[7]);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 8) tmem_dealloc(tmem_base, C::TMEM_COLS);
  if (p.KS > 1) {
    // merge: CTA `ks` of the cluster takes rows ks, ks + KS, ..; a warp per (row, panel)
    cluster_sync();
    const int mine = n_rows > ks ? (n_rows - ks + p.KS - 1) / p.KS : 0;
    for (int t = warp; t < mine * n_opan; t += LT_THREADS / 32) {
      const int r = ks + (t / n_opan) * p.KS, c = (t % n_opan) * 64 + lane * 2;
      const uint32_t base = smem_u32(reinterpret_cast<float*>(q_s) + r * C::OLD + c);
      float v0[LT_MAX_SPLITS], v1[LT_MAX_SPLITS], ms = -INFINITY, ls = 0.f;
#pragma unroll
      for (int q = 0; q < LT_MAX_SPLITS; ++q)
        if (q < p.KS) {
          const uint32_t rem = dsmem_map(base, (uint32_t)q);
          v0[q] = ld_dsmem_f32_at(rem);
          v1[q] = ld_dsmem_f32_at(rem + 4u);
        }
      if (lane < p.KS) {
        ls = ld_dsmem_f32(smem_u32(st_l + r), (uint32_t)lane);
        ms = ld_dsmem_f32(smem_u32(st_m + r), (uint32_t)lane);
      }
      const float snk = p.sink != nullptr ? p.sink[(row0 + r) % p.H] * LT_LOG2E : -INFINITY;
      const float mm = fmaxf(warp_max(ls > 0.f ? ms : -INFINITY), snk);
      float f = ls > 0.f ? exp2f(ms - mm) : 0.f;
      f *= 1.0f / (warp_sum(ls * f) + (p.sink != nullptr ? exp2f(snk - mm) : 0.f));
      float a0 = 0.f, a1 = 0.f;
#pragma unroll
      for (int q = 0; q < LT_MAX_SPLITS; ++q) {
        const float fq = __shfl_sync(0xffffffffu, f, q);
        if (q < p.KS && fq > 0.f) {                   // a split without keys for the row left nothing behind
          a0 = fmaf(fq, v0[q], a0);
          a1 = fmaf(fq, v1[q], a1);
        }
      }
      *reinterpret_cast<uint32_t*>(p.out + ((size_t)g_row0 + r) * p.ldc + vpan * 64 + c) = lt_pack(a0, a1);
    }
    cluster_sync();                                   // nobody leaves while its rows may still be read
  }
}

template <int NPAN>
static int latent_tc_launch(LatentTcParams& p, const CUtensorMap& tmC, const CUtensorMap& tmQ, cudaStream_t st) {
  using C = LtCfg<NPAN>;
  static bool configured = false;
  if (!configured) {
    CUDA_CHECK_RET(cudaFuncSetAttribute(latent_tc_kernel<NPAN>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM));
    configured = true;
  }
  cudaLaunchAttribute attr[2];
  int na = 0;
  if (p.pdl) {
    attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[na++].val.programmaticStreamSerializationAllowed = 1;
  }
  if (p.KS > 1) {
    attr[na].id = cudaLaunchAttributeClusterDimension;
    attr[na].val.clusterDim.x = 1;
    attr[na].val.clusterDim.y = (unsigned)p.KS;
    attr[na++].val.clusterDim.z = 1;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)(p.r.n_blk * p.MT * C::VSPLIT), (unsigned)p.KS);
  cfg.blockDim = dim3(LT_THREADS);
  cfg.dynamicSmemBytes = C::SMEM;
  cfg.stream = st;
  cfg.attrs = attr;
  cfg.numAttrs = na;
  CUDA_CHECK_RET(cudaLaunchKernelEx(&cfg, latent_tc_kernel<NPAN>, (const LatentTcParams)p, tmC, tmQ));
  return 0;
}

}  // namespace smc

// Largest padded latent width the tensor-core kernel takes.
SMC_API int smc_latent_tc_max_width() { return 512; }

// Key splits for `tiles` row tiles (blocks x 128-row tiles) over about `keys` cached rows: one wave of CTAs, at least
// LT_BK keys per split, powers of two so that a growing context re-plans rarely.
SMC_API int smc_latent_tc_splits(int tiles, int ldc, int keys) {
  const int v = ldc > 384 ? 2 : 1;
  int ks = 1;
  while (ks < smc::LT_MAX_SPLITS && (long long)tiles * v * ks * 2 <= 148 && keys / (ks * 2) >= smc::LT_BK) ks *= 2;
  return ks;
}

// a: as for smc_latent_attn (bf16).  tokens: query tokens in all; blk_rows: rows (tokens x heads) of the longest block;
// KS: key splits, at most eight.
SMC_API int smc_latent_attn_tc(const smc::LatentArgs* a, int tokens, int blk_rows, int KS, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_blk <= 0) return 0;
  if (a->ldc % 64 || a->ldc > 512 || KS < 1 || KS > LT_MAX_SPLITS) return -99;
  LatentTcParams p;
  p.pool = (const __nv_bfloat16*)a->pool; p.out = (__nv_bfloat16*)a->out;
  p.block_table = a->block_table; p.bt_stride = a->bt_stride; p.bt_rows = a->bt_rows; p.n_pages = a->n_pages;
  p.H = a->H; p.ldc = a->ldc; p.KS = KS; p.MT = (blk_rows + 127) / 128; p.T = tokens;
  p.scale_log2 = a->scale * LT_LOG2E;
  p.window = a->window; p.sink = a->sink;
  p.r = a->r; p.status = a->status; p.pdl = a->pdl;
  CUtensorMap tmC, tmQ;
  int rc = pool_tmap(&tmC, a->pool, (long long)a->n_pages + 1, a->ldc);
  if (rc == 0) rc = make_tmap(&tmQ, a->q, (long long)tokens * a->H, a->ldc, a->ldc, 128);
  if (rc) return rc;
  switch (a->ldc / 64) {
    case 1: return latent_tc_launch<1>(p, tmC, tmQ, st);
    case 2: return latent_tc_launch<2>(p, tmC, tmQ, st);
    case 3: return latent_tc_launch<3>(p, tmC, tmQ, st);
    case 4: return latent_tc_launch<4>(p, tmC, tmQ, st);
    case 5: return latent_tc_launch<5>(p, tmC, tmQ, st);
    case 6: return latent_tc_launch<6>(p, tmC, tmQ, st);
    case 7: return latent_tc_launch<7>(p, tmC, tmQ, st);
    case 8: return latent_tc_launch<8>(p, tmC, tmQ, st);
  }
  return -99;
}
