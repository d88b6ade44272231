// Tensor-map construction on the host and tiled copies (TMA) of bf16 operands into 128-byte-swizzled shared
// memory, with the matching tcgen05 operand descriptors. A copied box is 64 elements (128 bytes) wide; its rows
// follow one another, and every group of eight rows is one swizzle atom of 1024 bytes.
#pragma once

#include <cuda.h>
#include <cudaTypedefs.h>

#include "umma.cuh"

namespace leankv {
namespace tma {

constexpr int kBoxCols = 64;

// Map of a row-major bf16 tensor of `rank` dimensions (innermost first); strides in elements of dimensions 1 .. .
inline int make_map(CUtensorMap* map, const void* base, int rank, const cuuint64_t* dims, const cuuint64_t* strides,
                    const cuuint32_t* box) {
    static PFN_cuTensorMapEncodeTiled_v12000 encode = nullptr;
    if (encode == nullptr) {
        void* fn = nullptr;
        cudaDriverEntryPointQueryResult found;
        LEANKV_CUDA_TRY(cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &fn, 12000, cudaEnableDefault, &found));
        if (found != cudaDriverEntryPointSuccess || fn == nullptr) return LEANKV_EUNSUPPORTED;
        encode = reinterpret_cast<PFN_cuTensorMapEncodeTiled_v12000>(fn);
    }
    cuuint64_t bytes[4];
    cuuint32_t step[5] = {1, 1, 1, 1, 1};
    for (int i = 0; i + 1 < rank; ++i) bytes[i] = strides[i] * 2;
    const CUresult rc = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (cuuint32_t)rank, const_cast<void*>(base), dims, bytes,
                               box, step, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                               CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return rc == CUDA_SUCCESS ? LEANKV_OK : LEANKV_EINVAL;
}

__device__ __forceinline__ void expect(uint32_t bar, uint32_t bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
// x * 2 bytes must be a multiple of 16
__device__ __forceinline__ void load3(uint32_t dst, const CUtensorMap* map, int x, int y, int z, uint32_t bar) {
    asm volatile(
        "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];" ::"r"(dst),
        "l"(map), "r"(x), "r"(y), "r"(z), "r"(bar)
        : "memory");
}

// Descriptor of a swizzled operand: version 1 (bit 46), 128-byte swizzle (2 at bit 61). K-major: rows are M / N, eight-row
// groups 1024 bytes apart, a K = 16 step 32 bytes further inside the 128-byte row. MN-major: rows are K, the
// next eight rows 1024 bytes further, the next 64 columns `lead` bytes further.
__device__ __forceinline__ uint64_t swizzled(uint32_t addr, uint32_t lead) {
    return (uint64_t)((addr & 0x3FFFFu) >> 4) | ((uint64_t)(lead >> 4) << 16) | ((uint64_t)(1024u >> 4) << 32) | (1ull << 46) |
           (2ull << 61);
}
// D fp32 = A . B, both bf16, M = 128; B is K-major, or MN-major
__host__ __device__ constexpr uint32_t idesc_bf16(int n, bool b_mn) {
    return (1u << 4) | (1u << 7) | (1u << 10) | (b_mn ? 1u << 16 : 0u) | ((uint32_t)(n / 8) << 17) | (8u << 24);
}

}  // namespace tma
}  // namespace leankv
