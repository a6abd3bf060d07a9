// Hyper-connected residual streams and the short causal convolution of layered architectures.
//
//   hyper_step    one kernel between two sublayers: adds the finished sublayer's output to the streams
//                 (x_t <- sum_s mix[s][t] x_s + out[t] y), reads the next sublayer's input (u = sum_s in[s] x_s), divides
//                 it by its root mean square, applies the norm weight and hands it on in fp32 and / or in the activation
//                 type.  y may be a plain row or the weighted rows of a token's experts (plus the shared expert's).
//                 Its first form starts from the embedding (token row + learned position row, all streams equal), its
//                 last form ends with the plain sum of the streams.  With single-token sequences the short convolution
//                 of the next mixer is folded in: the history is one row of the state pool.
//   short_conv    the convolution on its own (several tokens per sequence): one thread per channel walks a block of
//                 tokens with the window in registers; the thread of a sequence's first block, which reads the old
//                 history, also writes the new one.
// Streams, norms and the convolution are computed in fp32.
#include "ragged.cuh"

namespace smc {

constexpr int HYPER_MAX_STREAMS = 16;
constexpr int HYPER_MAXV = 8;          // column groups per thread
constexpr int CONV_MAX_TAPS = 8;

struct HyperArgs {
  float* x;                       // [T, S, d]
  int S, d;
  // embedding start (ids != null) ...
  const int* ids;
  const int* positions;
  const void* embed;
  const void* pos;
  int vocab, max_pos;
  // ... or update with a sublayer's output
  const float* y;                 // [T, ldy] (null with experts only)
  int ldy;
  const float* ye;                // expert rows [slots, ldye]: y += sum_k route_w[t, k] * ye[route_slot[t, k]]
  int ldye, top;
  const int* route_slot;
  const float* route_w;
  const float* w_mix;             // [S, S] indexed [from][to]
  const float* w_out;             // [S]
  // next sublayer (w_in null: plain sum of the streams, nothing written back)
  const float* w_in;
  const float* norm_w;
  float eps;
  float* n_out;                   // fp32 normalised rows [T, d] (optional)
  void* xa;                       // activation rows [T, ldxa] (optional)
  int ldxa;
  // folded convolution (conv_w != null): token t is the only new token of the sequence with state row rows[t]
  const float* conv_w;            // [d, taps]
  float* hist;                    // [n_rows, d, taps - 1]
  const int* rows;
  int taps, n_rows;
  int* status;
  int pdl;
};

template <int VEC> struct Cols { float v[VEC]; };
template <int VEC, typename T> __device__ __forceinline__ Cols<VEC> ldc(const T* p) {
  Cols<VEC> r;
  if constexpr (VEC == 4) {
    const float4 a = load4(p);
    r.v[0] = a.x; r.v[1] = a.y; r.v[2] = a.z; r.v[3] = a.w;
  } else {
    r.v[0] = to_f32<T>(*p);
  }
  return r;
}
template <int VEC, typename T> __device__ __forceinline__ void stc(T* p, const Cols<VEC>& c) {
  if constexpr (VEC == 4) store4(p, make_float4(c.v[0], c.v[1], c.v[2], c.v[3]));
  else *p = from_f32<T>(c.v[0]);
}

// CONV: 0 no folded convolution, 1 taps and history in registers (up to 4 taps, two column groups per thread), 2 any.
constexpr int HYPER_CONV_GROUPS = 2, HYPER_CONV_HL = 3;

template <int S_T, typename AT, int VEC, int CONV>
__global__ void __launch_bounds__(CONV == 1 ? 512 : 256) hyper_step_kernel(const HyperArgs a) {
  constexpr int NV = CONV == 1 ? HYPER_CONV_GROUPS : HYPER_MAXV;
  __shared__ float red[32];
  __shared__ float s_mix[HYPER_MAX_STREAMS * HYPER_MAX_STREAMS], s_out[HYPER_MAX_STREAMS], s_in[HYPER_MAX_STREAMS];
  const int S = S_T > 0 ? S_T : a.S, d = a.d, t = blockIdx.x;
  constexpr int SM = S_T > 0 ? S_T : HYPER_MAX_STREAMS;
  // the coefficients are weights: they do not wait for the previous kernel
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) s_mix[i] = a.ids == nullptr ? a.w_mix[i] : 0.f;
  if (threadIdx.x < S) {
    s_out[threadIdx.x] = a.ids == nullptr ? a.w_out[threadIdx.x] : 0.f;
    s_in[threadIdx.x] = a.w_in != nullptr ? a.w_in[threadIdx.x] : 1.f;
  }
  constexpr int CG = CONV == 1 ? NV : 1, CH = CONV == 1 ? HYPER_CONV_HL : 1;
  float cw[CG][VEC][CH + 1], hv[CG][VEC][CH];
  const int hl = a.taps - 1;
  if constexpr (CONV == 1) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * VEC;
#pragma unroll
      for (int k = 0; k < VEC; ++k)
#pragma unroll
        for (int j = 0; j <= CH; ++j) cw[i][k][j] = (c < d && j <= hl) ? a.conv_w[(size_t)(c + k) * (hl + 1) + j] : 0.f;
    }
  }
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  int row = 0;
  if constexpr (CONV != 0) {
    row = a.rows[t];
    if (row < 0 || row >= a.n_rows) {
      if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
      row = -1;
    }
  }
  if constexpr (CONV == 1) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * VEC;
#pragma unroll
      for (int k = 0; k < VEC; ++k)
#pragma unroll
        for (int j = 0; j < CH; ++j)
          hv[i][k][j] = (c < d && j < hl && row >= 0) ? a.hist[((size_t)row * d + c + k) * hl + j] : 0.f;
    }
  }
  __syncthreads();
  float* x = a.x + (size_t)t * S * d;
  const AT *er = nullptr, *pr = nullptr;
  if (a.ids != nullptr) {
    int id = a.ids[t], p = a.positions[t];
    if (id < 0 || id >= a.vocab || p < 0 || p >= a.max_pos) {
      if (threadIdx.x == 0) atomicOr(a.status, SMC_ERR_BOUNDS);
      id = 0;
      p = 0;
    }
    er = reinterpret_cast<const AT*>(a.embed) + (size_t)id * d;
    pr = reinterpret_cast<const AT*>(a.pos) + (size_t)p * d;
  }
  const bool write_x = a.w_in != nullptr;
  Cols<VEC> u[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * VEC;
    if (c < d) {
      Cols<VEC> xs[SM], acc;
#pragma unroll
      for (int k = 0; k < VEC; ++k) acc.v[k] = 0.f;
      if (a.ids != nullptr) {
        const Cols<VEC> e = ldc<VEC>(er + c), p = ldc<VEC>(pr + c);
        Cols<VEC> v;
#pragma unroll
        for (int k = 0; k < VEC; ++k) v.v[k] = e.v[k] + p.v[k];
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < S) {
            if (write_x) stc<VEC>(x + (size_t)s * d + c, v);
#pragma unroll
            for (int k = 0; k < VEC; ++k) acc.v[k] = fmaf(s_in[s], v.v[k], acc.v[k]);
          }
      } else {
        Cols<VEC> y;
#pragma unroll
        for (int k = 0; k < VEC; ++k) y.v[k] = 0.f;
        if (a.y != nullptr) y = ldc<VEC>(a.y + (size_t)t * a.ldy + c);
        if (a.ye != nullptr)
          for (int k2 = 0; k2 < a.top; ++k2) {
            const float w = a.route_w[t * a.top + k2];
            const Cols<VEC> e = ldc<VEC>(a.ye + (size_t)a.route_slot[t * a.top + k2] * a.ldye + c);
#pragma unroll
            for (int k = 0; k < VEC; ++k) y.v[k] = fmaf(w, e.v[k], y.v[k]);
          }
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < S) xs[s] = ldc<VEC>(x + (size_t)s * d + c);
#pragma unroll
        for (int o = 0; o < SM; ++o)
          if (o < S) {
            Cols<VEC> v;
#pragma unroll
            for (int k = 0; k < VEC; ++k) v.v[k] = s_out[o] * y.v[k];
#pragma unroll
            for (int s = 0; s < SM; ++s)
              if (s < S) {
#pragma unroll
                for (int k = 0; k < VEC; ++k) v.v[k] = fmaf(s_mix[s * S + o], xs[s].v[k], v.v[k]);
              }
            if (write_x) stc<VEC>(x + (size_t)o * d + c, v);
#pragma unroll
            for (int k = 0; k < VEC; ++k) acc.v[k] = fmaf(s_in[o], v.v[k], acc.v[k]);
          }
      }
      u[i] = acc;
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss = fmaf(acc.v[k], acc.v[k], ss);
    }
  }
  const float inv = 1.0f / sqrtf(block_sum_all(ss, red) / (float)d + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * VEC;
    if (c < d) {
      const Cols<VEC> w = ldc<VEC>(a.norm_w + c);
      Cols<VEC> n;
#pragma unroll
      for (int k = 0; k < VEC; ++k) n.v[k] = u[i].v[k] * inv * w.v[k];
      if (a.n_out != nullptr) stc<VEC>(a.n_out + (size_t)t * d + c, n);
      if constexpr (CONV == 1) {
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
          float* hp = a.hist + ((size_t)max(row, 0) * d + c + k) * hl;
          float o = 0.f;
#pragma unroll
          for (int j = 0; j < CH; ++j) o = fmaf(cw[i][k][j], hv[i][k][j], o);      // zero beyond the history
#pragma unroll
          for (int j = 0; j <= CH; ++j)
            if (j == hl) o = fmaf(cw[i][k][j], n.v[k], o);
          if (row >= 0) {
#pragma unroll
            for (int j = 0; j < CH; ++j)
              if (j < hl) hp[j] = j + 1 < hl ? hv[i][k][j + 1 < CH ? j + 1 : j] : n.v[k];
            n.v[k] += o;
          }
        }
      }
      if (CONV == 2 && row >= 0) {
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
          const float* cw = a.conv_w + (size_t)(c + k) * a.taps;
          float* hp = a.hist + ((size_t)row * d + c + k) * hl;
          float o = cw[hl] * n.v[k];
          for (int j = 0; j < hl; ++j) {
            const float h = hp[j];
            o = fmaf(cw[j], h, o);
            if (j > 0) hp[j - 1] = h;
          }
          if (hl > 0) hp[hl - 1] = n.v[k];
          n.v[k] += o;
        }
      }
      if (a.xa != nullptr) stc<VEC>(reinterpret_cast<AT*>(a.xa) + (size_t)t * a.ldxa + c, n);
    }
  }
}

template <int TAPS, typename AT>
__global__ void __launch_bounds__(128) short_conv_kernel(const float* n, AT* xa, int ldxa,
                                                         const float* w, float* hist,
                                                         int n_rows, int d, const Ragged r, int* status, int pdl) {
  const int c = blockIdx.y * 128 + threadIdx.x;
  float wt[TAPS];
  if (c < d)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wt[j] = w[(size_t)c * TAPS + j];
  if (pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  if (c >= d) return;
  const RaggedBlock b = ragged_block(r, blockIdx.x);
  if (b.n <= 0) return;
  if (b.row < 0 || b.row >= n_rows) {
    if (threadIdx.x == 0) atomicOr(status, SMC_ERR_BOUNDS);
    return;
  }
  constexpr int HL = TAPS - 1;
  float* hp = hist + ((size_t)b.row * d + c) * HL;
  float old[HL > 0 ? HL : 1], win[HL > 0 ? HL : 1];      // win[j]: input of token start - HL + j
  const float* src = n + (size_t)b.off * d + c;
  if (b.start == 0) {
#pragma unroll
    for (int j = 0; j < HL; ++j) win[j] = old[j] = hp[j];
  } else {
#pragma unroll
    for (int j = 0; j < HL; ++j) win[j] = src[(ptrdiff_t)(b.start - HL + j) * d];   // B >= HL: always inside the sequence
  }
  for (int i = 0; i < b.n; ++i) {
    const float v = src[(size_t)(b.start + i) * d];
    float o = wt[HL] * v;
#pragma unroll
    for (int j = 0; j < HL; ++j) o = fmaf(wt[j], win[j], o);
    xa[(size_t)(b.off + b.start + i) * ldxa + c] = from_f32<AT>(v + o);
#pragma unroll
    for (int j = 0; j + 1 < HL; ++j) win[j] = win[j + 1];
    if (HL > 0) win[HL - 1] = v;
  }
  if (b.start == 0) {
    // last HL inputs of the sequence: new tokens where there are enough of them, else the tail of the old history
#pragma unroll
    for (int j = 0; j < HL; ++j) {
      const int t = b.len - HL + j;
      float v = 0.f;
      if (t >= 0) {
        v = src[(size_t)t * d];
      } else {
#pragma unroll
        for (int q = 0; q < HL; ++q)
          if (q == HL + t) v = old[q];
      }
      hp[j] = v;
    }
  }
}

template <int S_T, typename AT>
static int hyper_launch(const HyperArgs& a, int T, cudaStream_t st) {
  const bool vec = a.d % 4 == 0 && a.ldy % 4 == 0 && a.ldye % 4 == 0 && a.ldxa % 4 == 0;
  const int per = vec ? 4 : 1;
  const int groups = (a.d + per - 1) / per;
  int threads = groups <= 64 ? 64 : groups <= 128 ? 128 : 256;
  if (groups > threads * HYPER_MAXV) return -91;
#define SMC_HYPER(V, CV) return launch_pdl(hyper_step_kernel<S_T, AT, V, CV>, dim3(T), dim3(threads), 0, st, a.pdl, a)
  if (a.conv_w == nullptr) {
    if (vec) SMC_HYPER(4, 0);
    SMC_HYPER(1, 0);
  }
  if (vec && a.taps <= HYPER_CONV_HL + 1 && groups <= 512 * HYPER_CONV_GROUPS) {
    if (groups > threads * HYPER_CONV_GROUPS) threads = 512;
    SMC_HYPER(4, 1);
  }
  if (vec) SMC_HYPER(4, 2);
  SMC_HYPER(1, 2);
#undef SMC_HYPER
}

template <typename AT>
static int hyper_dispatch(const HyperArgs& a, int T, cudaStream_t st) {
  switch (a.S) {
    case 1: return hyper_launch<1, AT>(a, T, st);
    case 2: return hyper_launch<2, AT>(a, T, st);
    case 3: return hyper_launch<3, AT>(a, T, st);
    case 4: return hyper_launch<4, AT>(a, T, st);
  }
  return hyper_launch<0, AT>(a, T, st);
}

template <typename AT>
static int conv_dispatch(const float* n, AT* xa, int ldxa, const float* w, float* hist, int n_rows, int d, int taps,
                         const Ragged& r, int* status, int pdl, cudaStream_t st) {
  const dim3 grid(r.n_blk, (d + 127) / 128), block(128);
#define SMC_CONV(TP) \
  case TP: return launch_pdl(short_conv_kernel<TP, AT>, grid, block, 0, st, pdl, n, xa, ldxa, w, hist, n_rows, d, r, status, pdl);
  switch (taps) { SMC_CONV(1) SMC_CONV(2) SMC_CONV(3) SMC_CONV(4) SMC_CONV(5) SMC_CONV(6) SMC_CONV(7) SMC_CONV(8) }
#undef SMC_CONV
  return -92;
}

}  // namespace smc

SMC_API int smc_hyper_args_size() { return (int)sizeof(smc::HyperArgs); }
SMC_API int smc_ragged_size() { return (int)sizeof(smc::Ragged); }

// One step of the streams for T tokens (see HyperArgs); f32: embeddings and activations are fp32 instead of bf16.
SMC_API int smc_hyper_step(const smc::HyperArgs* a, int T, int f32, cudaStream_t st) {
  using namespace smc;
  if (T <= 0) return 0;
  if (a->S < 1 || a->S > HYPER_MAX_STREAMS || a->taps > 64) return -90;
  return f32 ? hyper_dispatch<float>(*a, T, st) : hyper_dispatch<__nv_bfloat16>(*a, T, st);
}

// h + conv(h) of the new tokens of every sequence: n fp32 [T, d] -> xa [T, ldxa]; hist [n_rows, d, taps - 1] advances.
SMC_API int smc_short_conv(const float* n, void* xa, int ldxa, const float* w, float* hist, int n_rows, int d, int taps,
                           const smc::Ragged* r, int* status, int f32, int pdl, cudaStream_t st) {
  using namespace smc;
  if (r->n_blk <= 0) return 0;
  if (r->B < taps - 1) return -93;
  if (f32) return conv_dispatch(n, (float*)xa, ldxa, w, hist, n_rows, d, taps, *r, status, pdl, st);
  return conv_dispatch(n, (__nv_bfloat16*)xa, ldxa, w, hist, n_rows, d, taps, *r, status, pdl, st);
}
