// Cached TMA tensor maps over bf16 matrices: a map is a pure function of address, extents and box, and encoding one is a
// driver call.
#pragma once
#include <map>
#include <mutex>
#include <tuple>

#include "tcgen05.cuh"

namespace ti {

struct AMapKey {
  const void* base;
  long long d0, d1;
  int b0, b1, swz;
  bool operator<(const AMapKey& o) const {
    return std::tie(base, d0, d1, b0, b1, swz) < std::tie(o.base, o.d0, o.d1, o.b0, o.b1, o.swz);
  }
};

// bf16 2-D tensor map [d1 rows][d0 columns] with row pitch d0 elements, box {b0, b1}; cached (an encode is a driver call)
inline int bf16_map_2d(CUtensorMap* dst, const void* base, long long d0, long long d1, int b0, int b1, CUtensorMapSwizzle swz) {
  static std::map<AMapKey, CUtensorMap> cache;
  static std::mutex mu;
  std::lock_guard<std::mutex> lock(mu);
  const AMapKey key{base, d0, d1, b0, b1, (int)swz};
  auto it = cache.find(key);
  if (it == cache.end()) {
    EncodeTiledFn enc = encode_tiled_fn();
    if (enc == nullptr) return 999;
    CUtensorMap m;
    const cuuint64_t dims[2] = {(cuuint64_t)d0, (cuuint64_t)d1};
    const cuuint64_t strides[1] = {(cuuint64_t)d0 * 2};
    const cuuint32_t box[2] = {(cuuint32_t)b0, (cuuint32_t)b1};
    const cuuint32_t elem[2] = {1, 1};
    const CUresult r = enc(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, elem,
                           CU_TENSOR_MAP_INTERLEAVE_NONE, swz, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return 1000 + (int)r;
    if (cache.size() > 4096) cache.clear();
    it = cache.emplace(key, m).first;
  }
  *dst = it->second;
  return 0;
}

// Rows of D columns seen as [groups of 8 rows][D/64 slabs][8 rows][64 columns], box `groups` x `slabs`: one copy brings
// whole 8-row groups with some of their column slabs side by side (for instance a 16-key cache page).
inline int bf16_map_groups(CUtensorMap* dst, const void* base, int D, long long rows, int slabs, int groups) {
  static std::map<AMapKey, CUtensorMap> cache;
  static std::mutex mu;
  std::lock_guard<std::mutex> lock(mu);
  const AMapKey key{base, D, rows, slabs, groups, -1};
  auto it = cache.find(key);
  if (it == cache.end()) {
    EncodeTiledFn enc = encode_tiled_fn();
    if (enc == nullptr) return 999;
    CUtensorMap m;
    const cuuint64_t dims[4] = {64, 8, (cuuint64_t)(D / 64), (cuuint64_t)(rows / 8)};
    const cuuint64_t strides[3] = {(cuuint64_t)D * 2, 128, (cuuint64_t)D * 16};
    const cuuint32_t box[4] = {64, 8, (cuuint32_t)slabs, (cuuint32_t)groups};
    const cuuint32_t elem[4] = {1, 1, 1, 1};
    const CUresult r = enc(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(base), dims, strides, box, elem,
                           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return 1000 + (int)r;
    if (cache.size() > 4096) cache.clear();
    it = cache.emplace(key, m).first;
  }
  *dst = it->second;
  return 0;
}

}  // namespace ti
