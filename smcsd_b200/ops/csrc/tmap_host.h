// Host-side helper: encode a 2-D bf16 tensor map (rows of 64 elements = 128 bytes per box row, SWIZZLE_128B),
// the layout every tcgen05 GEMM operand in this library is fetched with.
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>

#include <mutex>
#include <unordered_map>

namespace smc {

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

inline EncodeTiledFn get_encode_fn() {
  static EncodeTiledFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &ptr, 12000, cudaEnableDefault, &qres) ==
            cudaSuccess &&
        qres == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<EncodeTiledFn>(ptr);
  }
  return fn;
}

// bf16 matrix [rows, cols] row-major with leading dimension ld (elements); box = [box_rows, 64 cols].
// Reads outside [rows, cols] return zeros.
inline int make_tmap(CUtensorMap* tm, const void* base, long long rows, long long cols, long long ld, int box_rows) {
  EncodeTiledFn fn = get_encode_fn();
  if (!fn) return -1;
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
  cuuint32_t box[2] = {64u, (cuuint32_t)box_rows};
  cuuint32_t estr[2] = {1u, 1u};
  CUresult r = fn(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -2 - (int)r;
}

// 8-bit matrix [rows, cols] row-major with leading dimension ld (bytes); box = [box_rows, 128 bytes].
inline int make_tmap_u8(CUtensorMap* tm, const void* base, long long rows, long long cols, long long ld, int box_rows) {
  EncodeTiledFn fn = get_encode_fn();
  if (!fn) return -1;
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)ld};
  cuuint32_t box[2] = {128u, (cuuint32_t)box_rows};
  cuuint32_t estr[2] = {1u, 1u};
  CUresult r = fn(tm, CU_TENSOR_MAP_DATA_TYPE_UINT8, 2, const_cast<void*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -2 - (int)r;
}

// Tensor maps of page pools ([pages + 1, row] bf16, box = 64 columns x 64 pages), cached per pool.
struct PoolMapKey {
  const void* base; long long rows, cols;
  bool operator==(const PoolMapKey& o) const { return base == o.base && rows == o.rows && cols == o.cols; }
};
struct PoolMapHash {
  size_t operator()(const PoolMapKey& k) const {
    return std::hash<const void*>()(k.base) ^ (std::hash<long long>()(k.rows) * 1315423911u) ^ std::hash<long long>()(k.cols);
  }
};
inline int pool_tmap(CUtensorMap* tm, const void* base, long long rows, long long cols) {
  static std::unordered_map<PoolMapKey, CUtensorMap, PoolMapHash> cache;
  static std::mutex mu;
  std::lock_guard<std::mutex> lock(mu);
  const PoolMapKey key{base, rows, cols};
  auto it = cache.find(key);
  if (it != cache.end()) { *tm = it->second; return 0; }
  const int rc = make_tmap(tm, base, rows, cols, cols, 64);
  if (rc == 0) {
    if (cache.size() > 4096) cache.clear();
    cache.emplace(key, *tm);
  }
  return rc;
}

}  // namespace smc
