// Host-side creation of TMA tensor maps, shared by every kernel that loads operand tiles.
#include <cuda.h>
#include "scmx_gemm_core.cuh"

namespace scmx {

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static EncodeTiledFn encode_fn() {
    static EncodeTiledFn fn = nullptr;
    if (!fn) {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess &&
            q == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<EncodeTiledFn>(p);
    }
    return fn;
}

// Byte matrix [rows, row_bytes] with rows `pitch` bytes apart (0: row_bytes), box = box_bytes x box_rows, swizzle of 128 or 64
// bytes, zero fill outside.
int make_map_u8(CUtensorMap* map, const void* ptr, int64_t rows, int64_t row_bytes, int box_bytes, int box_rows, int swizzle_bytes,
                int64_t pitch) {
    EncodeTiledFn fn = encode_fn();
    SCMX_REQUIRE(fn != nullptr, SCMX_ECUDA, "cuTensorMapEncodeTiled is not available from this driver");
    const cuuint64_t dims[2] = {(cuuint64_t)row_bytes, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)(pitch ? pitch : row_bytes)};
    const cuuint32_t box[2] = {(cuuint32_t)box_bytes, (cuuint32_t)box_rows};
    const cuuint32_t estr[2] = {1, 1};
    const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_UINT8, 2, const_cast<void*>(ptr), dims, strides, box, estr,
                          CU_TENSOR_MAP_INTERLEAVE_NONE, swizzle_bytes == 64 ? CU_TENSOR_MAP_SWIZZLE_64B : CU_TENSOR_MAP_SWIZZLE_128B,
                          CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    SCMX_REQUIRE(r == CUDA_SUCCESS, SCMX_ECUDA, "cuTensorMapEncodeTiled failed with CUresult %d (rows=%lld row_bytes=%lld)", (int)r,
                 (long long)rows, (long long)row_bytes);
    return SCMX_OK;
}

// A stack of `planes` byte matrices [rows, row_bytes] (rows `pitch`, planes `plane_pitch` bytes apart, both multiples of 16), box =
// 128 bytes x box_rows of one plane, 128-byte swizzle, zero fill outside.
int make_map_planes(CUtensorMap* map, const void* ptr, int64_t planes, int64_t rows, int64_t row_bytes, int64_t pitch, int64_t plane_pitch,
                    int box_rows) {
    EncodeTiledFn fn = encode_fn();
    SCMX_REQUIRE(fn != nullptr, SCMX_ECUDA, "cuTensorMapEncodeTiled is not available from this driver");
    const cuuint64_t dims[3] = {(cuuint64_t)row_bytes, (cuuint64_t)rows, (cuuint64_t)planes};
    const cuuint64_t strides[2] = {(cuuint64_t)pitch, (cuuint64_t)plane_pitch};
    const cuuint32_t box[3] = {128, (cuuint32_t)box_rows, 1};
    const cuuint32_t estr[3] = {1, 1, 1};
    const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_UINT8, 3, const_cast<void*>(ptr), dims, strides, box, estr,
                          CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                          CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    SCMX_REQUIRE(r == CUDA_SUCCESS, SCMX_ECUDA, "cuTensorMapEncodeTiled failed with CUresult %d (planes=%lld rows=%lld row_bytes=%lld)", (int)r,
                 (long long)planes, (long long)rows, (long long)row_bytes);
    return SCMX_OK;
}

}  // namespace scmx
