// The driver's tensor-map encoder, looked up at run time (no link against libcuda).
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>

#include <mutex>

namespace kanso {

typedef CUresult (*TmEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*,
                               const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                               const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                               CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
inline TmEncodeFn tm_encoder() {
  static std::once_flag once;
  static TmEncodeFn fn = nullptr;
  std::call_once(once, [] {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) ==
            cudaSuccess &&
        q == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<TmEncodeFn>(p);
    else
      cudaGetLastError();
  });
  return fn;
}

// A 3-D map of bfloat16 rows: `cols` of `mid` rows, `stride1` elements apart, of `outer` records,
// `stride2` elements apart, read in boxes of 64 columns x box1 x box2.
inline bool tm_map3(TmEncodeFn encode, const void* base, uint64_t cols, uint64_t mid, uint64_t outer,
                 uint64_t stride1, uint64_t stride2, uint32_t box1, uint32_t box2,
                 CUtensorMap* map) {
  const cuuint64_t dim[3] = {cols, mid, outer};
  const cuuint64_t stride[2] = {stride1 * 2, stride2 * 2};
  const cuuint32_t box[3] = {64, box1, box2}, es[3] = {1, 1, 1};
  return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dim, stride, box,
                es, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// The same of plain rows: `rows` of `cols`, `ld` elements apart, in boxes of 64 columns x box rows.
inline bool tm_map2(TmEncodeFn encode, const void* base, uint64_t cols, uint64_t rows, uint64_t ld,
                    uint32_t box, CUtensorMap* map) {
  const cuuint64_t dim[2] = {cols, rows};
  const cuuint64_t stride[1] = {ld * 2};
  const cuuint32_t b[2] = {64, box}, es[2] = {1, 1};
  return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dim, stride, b,
                es, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

}  // namespace kanso
