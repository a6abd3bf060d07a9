// Residual stream of layers whose mixer and feed-forward run side by side on the same input.
//
//   side_step   one kernel between two layers: x <- x + s1 * mixer output + s2 * feed-forward output (scales per channel, or one
//               number for both; the mixer's may be a pair of rows, each under a norm of its own, of which half the sum counts;
//               the feed-forward's may be a plain row, a row times a gate per token, the weighted rows of the token's experts,
//               or both), the root mean square of the new row, and the row under two norms (weights per channel or a single
//               one): one operand for the next mixer, one for the next feed-forward (and in fp32 for its router).  Its first
//               form starts from the embedding, to which it may add a row chosen by the token and the one before it (kept in
//               the sequence's state between steps), and writes sine and cosine of the step's positions for all rotations of
//               the model; its last form hands on the row under the final norm alone.
// The stream, the scales, the gate and the norms are fp32.
#include "rotary.cuh"

namespace smc {

constexpr int SIDE_MAXV = 8;             // column groups per thread

struct SideArgs {
  float* x;                       // [T, d]
  int d;
  // embedding start (ids != null) ...
  const int* ids;
  const void* embed;              // [vocab, d]
  int vocab;
  float embed_scale;
  const void* pairs;              // [buckets + 1, d] rows of token pairs (optional): (before * mul_prev + id * mul_cur) mod buckets,
  int buckets;                    // the last row for a sequence's first token
  long long mul_prev, mul_cur;
  float* before;                  // row r: before[r * before_stride], the token before the first new one
  long long before_stride;
  int n_rows;
  Ragged r;                       // work list (with pairs)
  const int* positions;
  const double* freq;             // [n_freq] (optional)
  int n_freq;
  float2* angles;                 // [T, n_freq] {sine, cosine}
  // ... or update with the finished layer's outputs
  const float* y1;                // mixer [T, ldy]
  const float* s1;                // [d]
  const float* y2;                // feed-forward [T, ldy] (optional)
  const float* gate;              // [T] multiplies y2 (optional)
  int ldy;
  const float* ye;                // expert rows [slots, ldye] (optional): sum_k route_w[t, k] ye[route_slot[t, k]]
  int ldye, top;
  const int* route_slot;
  const float* route_w;
  const float* s2;                // [d]
  const float* yb;                // second mixer of a pair [T, ldy] (optional), norms of the two [d]
  const float* o1;
  const float* o2;
  float mult;                     // scale of both outputs where s1 is null
  float eps;
  const float* w1;                // norm of the next mixer (of the head with `final`) -> xa
  const float* w2;                // norm of the next feed-forward (optional) -> xb, n2
  int one_weight;                 // w1 and w2 are single numbers
  void* xa;                       // [T, ldxa]
  void* xb;
  float* n2;                      // [T, d] (optional)
  int ldxa;
  int final;                      // the stream itself is not written back
  int* status;
  int pdl;
};

// Sums of two values over the block.
__device__ __forceinline__ float2 block_sum_pair(float2 v, float2* red) {
  v.x = warp_sum(v.x);
  v.y = warp_sum(v.y);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  const float2 t = lane < nw ? red[lane] : make_float2(0.f, 0.f);
  return make_float2(warp_sum(t.x), warp_sum(t.y));
}

template <typename AT, int VEC, int NV, bool PAIR>
__global__ void __launch_bounds__(256) side_step_kernel(const SideArgs a) {
  __shared__ float red[32];
  const int d = a.d;
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  int t = blockIdx.x, id = 0, pair = 0, ends = -1;       // ends: the sequence's last new token, in the CTA of its first one
  float* keep = nullptr;
  if (a.pairs != nullptr) {
    const RaggedBlock b = ragged_block(a.r, blockIdx.x / a.r.B);
    const int i = blockIdx.x % a.r.B;
    if (i >= b.n) return;
    t = b.off + b.start + i;
    const int first = b.start + i == 0, p = b.prefix + b.start + i;
    int prev = first ? 0 : a.ids[t - 1];
    if (first) {
      if (b.row < 0 || b.row >= a.n_rows) {
        if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
      } else {
        keep = a.before + (size_t)b.row * a.before_stride;
        prev = (int)*keep;
        ends = b.off + b.len - 1;
      }
    }
    if (prev < 0 || prev >= a.vocab) prev = 0;             // reported where that token itself is looked up
    const int cur = min(max(a.ids[t], 0), a.vocab - 1);
    pair = p == 0 ? a.buckets : (int)((prev * a.mul_prev + cur * a.mul_cur) % a.buckets);
  }
  float* x = a.x + (size_t)t * d;
  float v[NV][VEC], ss = 0.f;
  if (a.ids != nullptr) {
    id = a.ids[t];
    if (id < 0 || id >= a.vocab) {
      if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
      id = 0;
    }
    if (a.freq != nullptr)
      for (int i = threadIdx.x; i < a.n_freq; i += blockDim.x) a.angles[(size_t)t * a.n_freq + i] = position_pair(a.freq, i, a.positions[t]);
  }
  const float gate = a.gate != nullptr ? a.gate[t] : 1.0f;
  float ya[PAIR ? NV : 1][VEC], yb[PAIR ? NV : 1][VEC];
  float2 unit = make_float2(1.f, 1.f);
  if constexpr (PAIR) {
    __shared__ float2 red2[32];
    float2 q = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * VEC;
      if (c >= d) continue;
      load_cols<VEC>(v[i], (const float*)x + c);
      load_cols<VEC>(ya[i], a.y1 + (size_t)t * a.ldy + c);
      load_cols<VEC>(yb[i], a.yb + (size_t)t * a.ldy + c);
#pragma unroll
      for (int k = 0; k < VEC; ++k) {
        q.x = fmaf(ya[i][k], ya[i][k], q.x);
        q.y = fmaf(yb[i][k], yb[i][k], q.y);
      }
    }
    q = block_sum_pair(q, red2);
    unit = make_float2(0.5f / sqrtf(q.x / (float)d + a.eps), 0.5f / sqrtf(q.y / (float)d + a.eps));
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * VEC;
    if (c >= d) continue;
    if (a.ids != nullptr) {
      load_cols<VEC>(v[i], reinterpret_cast<const AT*>(a.embed) + (size_t)id * d + c);
#pragma unroll
      for (int k = 0; k < VEC; ++k) v[i][k] *= a.embed_scale;
      if (a.pairs != nullptr) {
        float e[VEC];
        load_cols<VEC>(e, reinterpret_cast<const AT*>(a.pairs) + (size_t)pair * d + c);
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[i][k] += e[k];
      }
    } else {
      float y[VEC], s[VEC];
      if constexpr (PAIR) {
        float o[VEC];
        load_cols<VEC>(s, a.o1 + c);
        load_cols<VEC>(o, a.o2 + c);
#pragma unroll
        for (int k = 0; k < VEC; ++k) y[k] = fmaf(ya[i][k] * unit.x, s[k], yb[i][k] * unit.y * o[k]);
      } else {
        load_cols<VEC>(v[i], (const float*)x + c);
        load_cols<VEC>(y, a.y1 + (size_t)t * a.ldy + c);
      }
      if (a.s1 != nullptr) {
        load_cols<VEC>(s, a.s1 + c);
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[i][k] = fmaf(s[k], y[k], v[i][k]);
      } else {
        float f[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) f[k] = 0.f;
        if (a.y2 != nullptr) load_cols<VEC>(f, a.y2 + (size_t)t * a.ldy + c);
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[i][k] = fmaf(a.mult, y[k] + f[k], v[i][k]);
      }
      if (a.s2 != nullptr) {
        float f[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) f[k] = 0.f;
        if (a.y2 != nullptr) {
          load_cols<VEC>(y, a.y2 + (size_t)t * a.ldy + c);
#pragma unroll
          for (int k = 0; k < VEC; ++k) f[k] = gate * y[k];
        }
        if (a.ye != nullptr)
          for (int e = 0; e < a.top; ++e) {
            const float w = a.route_w[(size_t)t * a.top + e];
            load_cols<VEC>(y, a.ye + (size_t)a.route_slot[(size_t)t * a.top + e] * a.ldye + c);
#pragma unroll
            for (int k = 0; k < VEC; ++k) f[k] = fmaf(w, y[k], f[k]);
          }
        load_cols<VEC>(s, a.s2 + c);
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[i][k] = fmaf(s[k], f[k], v[i][k]);
      }
    }
    if (!a.final) store_cols<VEC>(x + c, v[i]);
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss = fmaf(v[i][k], v[i][k], ss);
  }
  const float inv = 1.0f / sqrtf(block_sum_all(ss, red) / (float)d + a.eps);
  if (ends >= 0 && threadIdx.x == 0) *keep = (float)a.ids[ends];        // every thread has read the old one
  const float g1 = a.one_weight ? a.w1[0] : 0.f, g2 = a.one_weight && a.w2 != nullptr ? a.w2[0] : 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * VEC;
    if (c >= d) continue;
    float w[VEC], o[VEC];
    if (a.one_weight) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) w[k] = g1;
    } else {
      load_cols<VEC>(w, a.w1 + c);
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) o[k] = v[i][k] * inv * w[k];
    store_cols<VEC>(reinterpret_cast<AT*>(a.xa) + (size_t)t * a.ldxa + c, o);
    if (a.w2 == nullptr) continue;
    if (a.one_weight) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) w[k] = g2;
    } else {
      load_cols<VEC>(w, a.w2 + c);
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) o[k] = v[i][k] * inv * w[k];
    store_cols<VEC>(reinterpret_cast<AT*>(a.xb) + (size_t)t * a.ldxa + c, o);
    if (a.n2 != nullptr) store_cols<VEC>(a.n2 + (size_t)t * d + c, o);
  }
}

template <typename AT>
static int side_launch(const SideArgs& a, int T, cudaStream_t st) {
  const bool vec = a.d % 4 == 0 && a.ldy % 4 == 0 && a.ldye % 4 == 0 && a.ldxa % 4 == 0;
  const int groups = vec ? a.d / 4 : a.d;
  const int threads = groups <= 64 ? 64 : groups <= 128 ? 128 : 256;
  if (groups > threads * SIDE_MAXV) return -91;
  const dim3 grid(a.pairs != nullptr ? a.r.n_blk * a.r.B : T), block(threads);
#define SMC_SIDE(VEC, NV)                                                                           \
  return a.yb != nullptr ? launch_pdl(side_step_kernel<AT, VEC, NV, true>, grid, block, 0, st, a.pdl, a) \
                         : launch_pdl(side_step_kernel<AT, VEC, NV, false>, grid, block, 0, st, a.pdl, a)
  if (!vec) SMC_SIDE(1, SIDE_MAXV);
  if (groups <= threads) SMC_SIDE(4, 1);
  if (groups <= threads * 2) SMC_SIDE(4, 2);
  SMC_SIDE(4, SIDE_MAXV);
#undef SMC_SIDE
}

}  // namespace smc

SMC_API int smc_side_args_size() { return (int)sizeof(smc::SideArgs); }

// One step of the stream for T tokens (see SideArgs); f32: embeddings and activations are fp32 instead of bf16.
SMC_API int smc_side_step(const smc::SideArgs* a, int T, int f32, cudaStream_t st) {
  using namespace smc;
  if (T <= 0) return 0;
  if (a->pairs != nullptr && (a->ids == nullptr || a->buckets < 1 || a->before == nullptr)) return -93;
  return f32 ? side_launch<float>(*a, T, st) : side_launch<__nv_bfloat16>(*a, T, st);
}
