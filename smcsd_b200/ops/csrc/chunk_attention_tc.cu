// Chunked or windowed attention of prompts in bf16: one CTA per (block of up to 64 tokens of a sequence, query head), four warps
// with 16 token rows each.  Keys run from the first one that the first token sees (the start of its chunk or window) to the last token in tiles of 64, gathered page by
// page with cp.async into two stages; scores and softmax stay in fp32 registers (base 2), P is rounded to bf16 for the
// second product and its sum is taken over the rounded values.  Chunk or window bound a CTA's work to a handful of tiles: the
// warp-level mma.sync products are short against the gather and the softmax, and a fragment layout in registers lets bias,
// mask, sink and gate be applied without a trip through tensor memory.
#include "chunk_attention.cuh"
#include "mma_sync.cuh"

namespace smc {

constexpr int CT_Q = 64, CT_K = 64;

// 64 rows of `cols` bf16 values into [64][W * 16 + 8], zeros beyond; row i comes from src + index(i) * ld (index < 0: zeros).
template <int W, typename F>
__device__ __forceinline__ void gather_tile(__nv_bfloat16* dst, const __nv_bfloat16* src, size_t ld, int cols, F index) {
  for (int x = threadIdx.x; x < 64 * W * 2; x += 128) {
    const int i = x / (W * 2), c = (x - i * W * 2) * 8;
    const int at = index(i);
    const bool real = at >= 0 && c < cols;
    cp_async16(smem_u32(dst + i * (W * 16 + 8) + c), real ? src + (size_t)at * ld + c : src, real);
  }
}

template <int ND, int NV>
__global__ void __launch_bounds__(128) chunk_attn_tc_kernel(const ChunkAttnArgs a) {
  constexpr int LD = ND * 16 + 8, LV = NV * 16 + 8;
  extern __shared__ __align__(16) uint8_t ct_smem[];
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(ct_smem);
  __nv_bfloat16* sk = sq + CT_Q * LD;
  __nv_bfloat16* sv = sk + 2 * CT_K * LD;
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  const RaggedBlock b = ragged_block(a.r, blockIdx.x);
  if (b.n <= 0) return;
  if (b.row < 0 || b.row >= a.bt_rows || b.prefix < 0 || b.prefix + b.len > a.bt_stride) {
    if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, g = h / (a.H / a.G);
  const int p0 = b.prefix + b.start, t0 = b.off + b.start, k_begin = first_key(a, p0), k_end = p0 + b.n;
  const int* bt = a.block_table + (size_t)b.row * a.bt_stride;
  const __nv_bfloat16* kp = reinterpret_cast<const __nv_bfloat16*>(a.kpool) + (size_t)g * a.D;
  const __nv_bfloat16* vp = reinterpret_cast<const __nv_bfloat16*>(a.vpool) + (size_t)g * a.V;
  auto page_of = [&](int k) {
    if (k >= k_end) return -1;
    const int p = bt[k];
    if (p < 0 || p > a.n_pages) { atomicOr(a.status, SMC_ERR_BOUNDS); return -1; }
    return p;
  };
  auto fetch = [&](int tile, int st) {
    const int k0 = k_begin + tile * CT_K;
    auto at = [&](int i) { return page_of(k0 + i); };
    gather_tile<ND>(sk + st * CT_K * LD, kp, (size_t)a.G * a.D, a.D, at);
    gather_tile<NV>(sv + st * CT_K * LV, vp, (size_t)a.G * a.V, a.V, at);
  };
  gather_tile<ND>(sq, reinterpret_cast<const __nv_bfloat16*>(a.q) + ((size_t)t0 * a.H + h) * a.D, (size_t)a.H * a.D, a.D,
                  [&](int i) { return i < b.n ? i : -1; });
  const int n_tiles = (k_end - k_begin + CT_K - 1) / CT_K;
  fetch(0, 0);
  cp_async_commit();
  const float sc = a.scale * 1.4426950408889634f;
  const float cap = a.softcap * 1.4426950408889634f, cap_in = a.softcap > 0.f ? 2.0f / a.softcap : 0.f;
  const float r1 = a.r1 != nullptr ? a.r1[h] : 0.f, r2 = a.r1 != nullptr ? a.r2[h] : 0.f;
  const int row0 = warp * 16 + (lane >> 2);                // this thread's rows: row0 and row0 + 8
  const int pos[2] = {p0 + row0, p0 + row0 + 8};
  const int lo[2] = {first_key(a, pos[0]), first_key(a, pos[1])};
  const bool active = warp * 16 < b.n;
  const int w_lo = first_key(a, p0 + warp * 16), w_hi = p0 + warp * 16 + 15;
  float o[NV * 2][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int j = 0; j < NV * 2; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
  const uint32_t q_addr = smem_u32(sq + (warp * 16 + (lane & 15)) * LD + (lane >> 4) * 8);
  const int kr = (lane & 7) + ((lane >> 4) << 3), kc = ((lane >> 3) & 1) * 8;      // K: key row and dim column of a 16 x 16 block
  const int vr = lane & 15, vc = (lane >> 4) * 8;                                  // V: key row and value column
  for (int tile = 0; tile < n_tiles; ++tile) {
    const int st = tile & 1, k0 = k_begin + tile * CT_K;
    if (tile + 1 < n_tiles) fetch(tile + 1, st ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    if (active && k0 <= w_hi && k0 + CT_K > w_lo) {
      float s[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
      const uint32_t k_addr = smem_u32(sk + st * CT_K * LD + kr * LD + kc);
#pragma unroll
      for (int kd = 0; kd < ND; ++kd) {
        uint32_t qa[4];
        ldsm4(qa, q_addr + kd * 32);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          uint32_t kb[4];
          ldsm4(kb, k_addr + j * 16 * LD * 2 + kd * 32);
          mma16816(s[2 * j], qa, kb[0], kb[1]);
          mma16816(s[2 * j + 1], qa, kb[2], kb[3]);
        }
      }
      float top[2] = {m[0], m[1]};
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = e >> 1, key = k0 + j * 8 + (lane & 3) * 2 + (e & 1);
          float v = s[j][e] * sc;
          if (a.softcap > 0.f) v = cap * (1.0f - __fdividef(2.0f, 1.0f + exp2f(v * cap_in)));     // cap tanh
          if (a.r1 != nullptr) v = fmaf(-r1, __log2f(fmaf(r2, (float)max(pos[r] - key, 0), 1.0f)), v);
          v = (key > pos[r] || key < lo[r]) ? -INFINITY : v;
          s[j][e] = v;
          top[r] = fmaxf(top[r], v);
        }
      float base[2], f[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        top[r] = fmaxf(top[r], __shfl_xor_sync(0xffffffffu, top[r], 1));
        top[r] = fmaxf(top[r], __shfl_xor_sync(0xffffffffu, top[r], 2));
        base[r] = top[r] == -INFINITY ? 0.f : top[r];          // no key seen yet
        f[r] = exp2f(m[r] - base[r]);
        m[r] = top[r];
        l[r] *= f[r];
      }
#pragma unroll
      for (int j = 0; j < NV * 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] *= f[e >> 1];
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t pa[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {                          // {rows, rows + 8} x {keys 0-7, keys 8-15}
          const int j = kk * 2 + (x >> 1), r = x & 1;
          const __nv_bfloat162 pp = __floats2bfloat162_rn(exp2f(s[j][r * 2] - base[r]), exp2f(s[j][r * 2 + 1] - base[r]));
          l[r] += __low2float(pp) + __high2float(pp);
          pa[x] = *reinterpret_cast<const uint32_t*>(&pp);
        }
        const uint32_t v_addr = smem_u32(sv + st * CT_K * LV + (kk * 16 + vr) * LV + vc);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          uint32_t vb[4];
          ldsm4_t(vb, v_addr + j * 32);
          mma16816(o[2 * j], pa, vb[0], vb[1]);
          mma16816(o[2 * j + 1], pa, vb[2], vb[3]);
        }
      }
    }
    __syncthreads();
  }
  cp_async_wait<0>();
  if (!active) return;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int row = row0 + r * 8;
    if (row >= b.n) continue;
    const float extra = a.sink_logit != nullptr ? a.sink_logit[h] * 1.4426950408889634f : 0.f;
    const float mm = a.sink ? fmaxf(m[r], extra) : m[r];
    const float f = exp2f(m[r] - mm), inv = f / (l[r] * f + (a.sink ? exp2f(extra - mm) : 0.f));
    const size_t at = (size_t)(t0 + row) * a.H * a.V + (size_t)h * a.V;
    const float* gate = a.gate != nullptr ? a.gate + (size_t)(t0 + row) * a.ldg + (a.gate_heads ? h : h * a.V) : nullptr;
    const float head_gate = gate != nullptr && a.gate_heads ? 1.0f / (1.0f + __expf(-gate[0])) : 1.0f;
#pragma unroll
    for (int j = 0; j < NV * 2; ++j) {
      const int c = j * 8 + (lane & 3) * 2;
      if (c >= a.V) continue;
      const float2 back = turn_back(a, t0 + row, c, make_float2(o[j][r * 2] * inv, o[j][r * 2 + 1] * inv));
      float v0 = back.x, v1 = back.y;
      if (a.gate_heads) {
        v0 *= head_gate;
        v1 *= head_gate;
      } else if (gate != nullptr) {
        v0 /= 1.0f + __expf(-gate[c]);
        v1 /= 1.0f + __expf(-gate[c + 1]);
      }
      *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<__nv_bfloat16*>(a.out) + at + c) = __floats2bfloat162_rn(v0, v1);
    }
  }
}

template <int ND, int NV>
static int chunk_tc_launch(const ChunkAttnArgs& a, cudaStream_t st) {
  constexpr int bytes = (3 * 64 * (ND * 16 + 8) + 2 * 64 * (NV * 16 + 8)) * 2;
  CUDA_CHECK_RET(cudaFuncSetAttribute(chunk_attn_tc_kernel<ND, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
  return launch_pdl(chunk_attn_tc_kernel<ND, NV>, dim3(a.r.n_blk, a.H), dim3(128), bytes, st, a.pdl, a);
}

template <int ND>
static int chunk_tc_values(const ChunkAttnArgs& a, cudaStream_t st) {
  if (a.V <= 32) return chunk_tc_launch<ND, 2>(a, st);
  if (a.V <= 64) return chunk_tc_launch<ND, 4>(a, st);
  if (a.V <= 128) return chunk_tc_launch<ND, 8>(a, st);
  return chunk_tc_launch<ND, 16>(a, st);
}

}  // namespace smc

SMC_API int smc_chunk_attn_tc_max_width() { return 256; }

// The same step in bf16 for blocks of up to 64 tokens (r.B <= 64).
SMC_API int smc_chunk_attn_tc(const smc::ChunkAttnArgs* a, cudaStream_t st) {
  using namespace smc;
  if (a->r.n_blk <= 0) return 0;
  if (a->D % 8 || a->V % 8 || a->H % a->G || (a->chunk < 1 && a->window < 1) || a->turn % 2 || a->r.B > CT_Q || a->D > 256 || a->V > 256) return -110;
  if (a->D <= 32) return chunk_tc_values<2>(*a, st);
  if (a->D <= 64) return chunk_tc_values<4>(*a, st);
  if (a->D <= 128) return chunk_tc_values<8>(*a, st);
  return chunk_tc_values<16>(*a, st);
}
