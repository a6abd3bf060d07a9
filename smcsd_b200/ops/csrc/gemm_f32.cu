// fp32 GEMM on the CUDA cores (no tensor-core rounding) for models that run in 32-bit: Y[m, n] = sum_k X[m, k] W[n, k].
// Same grouped forms as the tensor-core GEMM: one product, one per group of weight rows and column ranges ("batched"), or
// token tiles taken from a table in device memory ("tiled").  64 x 64 tiles, sixteen outputs per thread.
#include "ragged.cuh"

namespace smc {

constexpr int F32_TILE = 64, F32_BK = 16;

struct GemmF32Args {
  const float* W;           // [groups * w_rows.., K]
  const float* X;           // [M, ldx]
  float* out;               // [M, ldo]
  int N, K, M, ldx, ldo;
  int mode, groups, w_rows, x_cols, out_cols;
  const int4* tiles;        // {group, first row, end row, -}, at most F32_TILE rows each
  int relu2;                // out = max(., 0)^2
  int pdl;
};

__global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32Args a) {
  __shared__ float sx[F32_BK][F32_TILE + 4], sw[F32_BK][F32_TILE + 4];
  if (a.pdl) { pdl_launch_dependents(); pdl_wait_prior_grid(); }
  int g = 0, m0, m_lim = a.M;
  if (a.mode == 2) {
    const int4 t = a.tiles[blockIdx.y];
    g = t.x; m0 = t.y; m_lim = t.z;
    if (g < 0 || g >= a.groups || m0 < 0 || m0 >= m_lim || m_lim > a.M) return;
  } else {
    m0 = blockIdx.y * F32_TILE;
    if (a.mode == 1) g = blockIdx.z;
  }
  const int n0 = blockIdx.x * F32_TILE;
  const float* W = a.W + (size_t)g * a.w_rows * a.K;
  const float* X = a.X + (a.mode == 1 ? (size_t)g * a.x_cols : 0);
  float* out = a.out + (a.mode == 1 ? (size_t)g * a.out_cols : 0);
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;       // 4 weight rows x 4 tokens each
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += F32_BK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = ty + i * 16, k = k0 + tx;
      sx[tx][r] = (m0 + r < m_lim && k < a.K) ? X[(size_t)(m0 + r) * a.ldx + k] : 0.f;
      sw[tx][r] = (n0 + r < a.N && k < a.K) ? W[(size_t)(n0 + r) * a.K + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < F32_BK; ++k) {
      float xv[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { xv[i] = sx[k][ty * 4 + i]; wv[i] = sw[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      const float v = a.relu2 ? fmaxf(acc[i][j], 0.f) * fmaxf(acc[i][j], 0.f) : acc[i][j];
      if (m < m_lim && n < a.N) out[(size_t)m * a.ldo + n] = v;
    }
}

}  // namespace smc

// mode 0: one product; 1: batched over groups; 2: tiled (max_tiles table entries of at most 64 rows).  relu2: squared relu on top.
SMC_API int smc_gemm_f32(const float* W, const float* X, float* out, int N, int K, int M, int ldx, int ldo, int mode,
                         int groups, int w_rows, int x_cols, int out_cols, const int4* tiles, int max_tiles, int relu2,
                         int pdl, cudaStream_t st) {
  using namespace smc;
  if (M <= 0 || N <= 0) return 0;
  if (mode == 2 && (tiles == nullptr || max_tiles < 1)) return -32;
  GemmF32Args a{W, X, out, N, K, M, ldx, ldo, mode, groups, w_rows, x_cols, out_cols, tiles, relu2, pdl};
  const int mt = mode == 2 ? max_tiles : (M + F32_TILE - 1) / F32_TILE;
  if (mt > 65535) return -35;
  return launch_pdl(gemm_f32_kernel, dim3((N + F32_TILE - 1) / F32_TILE, mt, mode == 1 ? groups : 1), dim3(256), 0, st, pdl, a);
}
