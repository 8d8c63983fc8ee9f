// Tensor-map descriptors of cache tensors for the kernels that fetch cache rows by the TMA unit.
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>
#include <map>
#include <mutex>
#include <tuple>

namespace ts {

typedef CUresult (*DtEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                               const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                               CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static DtEncodeFn dt_encode_fn() {
  static DtEncodeFn fn = nullptr;
  if (fn == nullptr) {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess &&
        q == cudaDriverEntryPointSuccess)
      fn = (DtEncodeFn)p;
  }
  return fn;
}

// The descriptor of one cache tensor ([rows, head_dim] bf16, boxes of box_rows x 64, 128-byte
// swizzle). Descriptors are kept per (address, rows, head_dim, box_rows): a cache tensor is
// allocated once and used for every step.
static const CUtensorMap* cache_map(const void* base, long long rows, int head_dim, int box_rows) {
  static std::mutex mu;
  static std::map<std::tuple<const void*, long long, int, int>, CUtensorMap> maps;
  std::lock_guard<std::mutex> lock(mu);
  auto key = std::make_tuple(base, rows, head_dim, box_rows);
  auto it = maps.find(key);
  if (it != maps.end()) return &it->second;
  DtEncodeFn fn = dt_encode_fn();
  if (fn == nullptr) return nullptr;
  CUtensorMap m;
  cuuint64_t dims[2] = {(cuuint64_t)head_dim, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)head_dim * 2};
  cuuint32_t box[2] = {64u, (cuuint32_t)box_rows};
  cuuint32_t elem[2] = {1, 1};
  if (fn(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, elem,
         CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
         CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return nullptr;
  return &maps.emplace(key, m).first->second;
}

// The same tensor seen as [pages * kv_heads, page_size, head_dim], boxes of box_heads x box_rows x 64 columns: the same
// rows of several key/value heads of a page in one copy.
static const CUtensorMap* cache_heads_map(const void* base, long long page_heads, int page_size, int head_dim, int box_rows, int box_heads) {
  static std::mutex mu;
  static std::map<std::tuple<const void*, long long, int, int, int, int>, CUtensorMap> maps;
  std::lock_guard<std::mutex> lock(mu);
  auto key = std::make_tuple(base, page_heads, page_size, head_dim, box_rows, box_heads);
  auto it = maps.find(key);
  if (it != maps.end()) return &it->second;
  DtEncodeFn fn = dt_encode_fn();
  if (fn == nullptr) return nullptr;
  CUtensorMap m;
  cuuint64_t dims[3] = {(cuuint64_t)head_dim, (cuuint64_t)page_size, (cuuint64_t)page_heads};
  cuuint64_t strides[2] = {(cuuint64_t)head_dim * 2, (cuuint64_t)head_dim * 2 * page_size};
  cuuint32_t box[3] = {64u, (cuuint32_t)box_rows, (cuuint32_t)box_heads};
  cuuint32_t elem[3] = {1, 1, 1};
  if (fn(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, elem,
         CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
         CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return nullptr;
  return &maps.emplace(key, m).first->second;
}

}  // namespace ts
