// Work list of one model step over sequences of unequal length: every sequence brings a run of new tokens that continue
// what the cache and the state already hold.  Kernels walk the list in blocks of at most B consecutive tokens of one
// sequence.  Two forms share it: explicit device arrays (prompts, portions of prompts and single tokens side by side), or,
// with null block arrays, a uniform batch of n_seq sequences with E tokens each (what a captured decode step uses).
#pragma once
#include "common.cuh"

namespace smc {

struct Ragged {
  const int* seq_row;       // [n_seq] block-table / state row
  const int* seq_prefix;    // [n_seq] tokens already held
  const int* seq_off;       // [n_seq] first token of the sequence in this step (null: uniform)
  const int* seq_len;       // [n_seq] new tokens (null: uniform)
  const int* blk_seq;       // [n_blk] (null: uniform)
  const int* blk_start;     // [n_blk] first token of the block, relative to the sequence's first new token
  int n_seq, n_blk, E, B;
};

struct RaggedBlock {
  int row, prefix;          // of the sequence
  int off, len;             // of the sequence's new tokens in this step
  int start, n;             // this block: tokens [off + start, off + start + n)
};

__device__ __forceinline__ RaggedBlock ragged_block(const Ragged& r, int blk) {
  RaggedBlock b;
  int s;
  if (r.blk_seq != nullptr) {
    s = r.blk_seq[blk];
    b.start = r.blk_start[blk];
    b.off = r.seq_off[s];
    b.len = r.seq_len[s];
  } else {
    const int per = (r.E + r.B - 1) / r.B;
    s = blk / per;
    b.start = (blk - s * per) * r.B;
    b.off = s * r.E;
    b.len = r.E;
  }
  b.row = r.seq_row[s];
  b.prefix = r.seq_prefix[s];
  b.n = min(r.B, b.len - b.start);
  return b;
}

// Activation element types: bf16 on the serving path, fp32 for 32-bit runs.
template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// Four consecutive elements.
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
  return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 o;
  o.x = *reinterpret_cast<uint32_t*>(&a);
  o.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = o;
}

// VEC (1 or 4) consecutive elements.
template <int VEC, typename T> __device__ __forceinline__ void load_cols(float (&v)[VEC], const T* p) {
  if constexpr (VEC == 4) {
    const float4 a = load4(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  } else {
    v[0] = to_f32<T>(*p);
  }
}
template <int VEC, typename T> __device__ __forceinline__ void store_cols(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) store4(p, make_float4(v[0], v[1], v[2], v[3]));
  else *p = from_f32<T>(v[0]);
}

__device__ __forceinline__ float block_sum_all(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  const float t = warp_sum(lane < nw ? red[lane] : 0.f);
  __syncthreads();
  return t;
}

// Launch with an optional programmatic dependency on the previous kernel of the stream.  Kernels launched this way take
// data of earlier kernels through plain pointers: a const __restrict__ parameter counts as invariant for the compiler, which
// may then read it ahead of the wait.
// launch_cluster: the same with `cluster` consecutive CTAs in x as a thread-block cluster.
template <typename... P, typename... A>
inline int launch_cluster(void (*kern)(P...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, int pdl, int cluster, A... args) {
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (pdl) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n++].val.programmaticStreamSerializationAllowed = 1;
  }
  if (cluster > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = cluster;
    attr[n].val.clusterDim.y = 1;
    attr[n++].val.clusterDim.z = 1;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cfg.attrs = attr;
  cfg.numAttrs = n;
  CUDA_CHECK_RET(cudaLaunchKernelEx(&cfg, kern, static_cast<P>(args)...));
  return 0;
}
template <typename... P, typename... A>
inline int launch_pdl(void (*kern)(P...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, int pdl, A... args) {
  return launch_cluster(kern, grid, block, smem, st, pdl, 1, args...);
}

}  // namespace smc
