// Host side of the TMA loads: tensor maps over [batch, rows, heads, d] tensors.
#pragma once
#include <cuda.h>

#include "common.cuh"

namespace sk {

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

inline EncodeTiledFn encode_tiled_fn() {
    static EncodeTiledFn fn = nullptr;
    if (fn == nullptr) {
        void* f = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &f, cudaEnableDefault, &q) == cudaSuccess &&
            q == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<EncodeTiledFn>(f);
    }
    return fn;
}

// [batch, rows, heads, d] bf16 with a contiguous last dimension -> boxes of box_rows rows x 64 columns of one head,
// 128-byte swizzle; what lies outside the tensor reads as zero
inline int make_head_map(CUtensorMap* map, const void* base, int d, int heads, int64_t rows, int batch, int64_t hs, int64_t rs,
                         int64_t bs, int box_rows) {
    EncodeTiledFn enc = encode_tiled_fn();
    if (enc == nullptr) return fail(SK_ERR_CUDA, "skb_attn: cuTensorMapEncodeTiled is not available");
    if (batch == 1) bs = rs;                                  // never stepped over
    if (heads == 1) hs = rs;
    const cuuint64_t dims[4] = {(cuuint64_t)d, (cuuint64_t)heads, (cuuint64_t)rows, (cuuint64_t)batch};
    const cuuint64_t strides[3] = {(cuuint64_t)hs * 2, (cuuint64_t)rs * 2, (cuuint64_t)bs * 2};
    const cuuint32_t box[4] = {64, 1, (cuuint32_t)box_rows, 1};
    const cuuint32_t estr[4] = {1, 1, 1, 1};
    const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(base), dims, strides, box, estr,
                           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(SK_ERR_CUDA, "skb_attn: cuTensorMapEncodeTiled failed (%d)", (int)r);
    return SK_OK;
}

inline bool head_map_ok(const void* base, int d, int64_t hs, int64_t rs, int64_t bs) {
    return (uintptr_t)base % 16 == 0 && d % 8 == 0 && hs % 8 == 0 && rs % 8 == 0 && bs % 8 == 0;
}

}  // namespace sk
