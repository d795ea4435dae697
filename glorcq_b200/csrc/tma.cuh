// Tensor maps and tiled TMA loads (no multicast) of bfloat16 operands in the 128-byte swizzle that the tcgen05
// descriptors of tc_mm.cuh describe.
#pragma once

#include <cuda.h>

#include "dense_common.cuh"

namespace glq {

typedef CUresult (*EncodeTiled)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
inline EncodeTiled encode_tiled() {
    static EncodeTiled fn = [] {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult st;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &st) != cudaSuccess ||
            st != cudaDriverEntryPointSuccess)
            p = nullptr;
        return reinterpret_cast<EncodeTiled>(p);
    }();
    return fn;
}
// `rank` dimensions, innermost first; strides in elements of dimensions 1..; the innermost box is 64 wide; zeros outside.
// Base and strides are multiples of 16 bytes.
inline bool make_map_nd(CUtensorMap* m, const void* base, int rank, const long* size, const long* stride, const int* box) {
    cuuint64_t dims[3], st[2];
    cuuint32_t bx[3], es[3] = {1, 1, 1};
    for (int i = 0; i < rank; ++i) {
        dims[i] = (cuuint64_t)size[i];
        bx[i] = (cuuint32_t)box[i];
        if (i) st[i - 1] = (cuuint64_t)stride[i] * 2;
    }
    return encode_tiled()(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void*>(base), dims, st, bx, es,
                          CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                          CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}
// (rows, K) with row stride ld; boxes of 64 columns x box_rows
inline bool make_map(CUtensorMap* m, const void* base, long rows, long K, long ld, int box_rows) {
    const long size[2] = {K, rows}, stride[2] = {1, ld};
    const int box[2] = {64, box_rows};
    return make_map_nd(m, base, 2, size, stride, box);
}

__device__ __forceinline__ void tma_load_2d(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst),
        "l"(map), "r"(x), "r"(y), "r"(bar)
        : "memory");
}
__device__ __forceinline__ void tma_load_3d(uint32_t dst, const CUtensorMap* map, int x, int y, int z, uint32_t bar) {
    asm volatile(
        "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];" ::"r"(dst),
        "l"(map), "r"(x), "r"(y), "r"(z), "r"(bar)
        : "memory");
}
// bf16 operands, both K-major, fp32 accumulator, M = 128
__host__ __device__ constexpr uint32_t dt_idesc(int n) { return tc_idesc(n) | (1u << 7) | (1u << 10); }
// tc_wait of all lanes of a warp, with one answer
__device__ __forceinline__ bool tc_wait_warp(uint32_t bar, uint32_t parity, volatile int* dead, int code) {
    return __all_sync(0xffffffffu, tc_wait(bar, parity, dead, code));
}

}  // namespace glq
