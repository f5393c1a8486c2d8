// Host side of the tensor-core GEMMs of prefill.cuh, shared by the families' prompt passes: tensor maps and launches.
#pragma once
#include "prefill.cuh"

#include "model.h"

namespace cd {
namespace {

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

inline EncodeTiledFn encode_tiled_fn() {  // nullptr: this driver does not have it
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres) != cudaSuccess || qres != cudaDriverEntryPointSuccess) return nullptr;
    return (EncodeTiledFn)fn;
}

inline size_t round_up(size_t v, size_t a) { return (v + a - 1) / a * a; }

bool encode_2d(EncodeTiledFn encode, CUtensorMap* map, CUtensorMapDataType dt, const void* base, uint64_t inner, uint64_t rows,
               uint64_t row_bytes, uint32_t box_rows) {
    const cuuint64_t dims[2] = {inner, rows};
    const cuuint64_t strides[1] = {row_bytes};
    const cuuint32_t box[2] = {(cuuint32_t)PF_BK, box_rows};
    const cuuint32_t estr[2] = {1, 1};
    return encode(map, dt, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                     CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// instruction descriptor of tcgen05.mma kind::f16: fp32 accumulate, both operands K-major, M = 128
inline uint32_t make_idesc(int bn, bool bf16) {
    const uint32_t fmt = bf16 ? 1u : 0u;
    return (1u << 4) | (fmt << 7) | (fmt << 10) | ((uint32_t)(bn >> 3) << 17) | ((uint32_t)(PF_BM >> 4) << 24);
}

template <int BN, bool SPLIT, class Epi>
cudaError_t pf_launch_t(cd_model* m, const CUtensorMap& a, const CUtensorMap& a_lo, const CUtensorMap& b, const PfGemm& p, bool bf16, int zdim,
                        const Epi& epi) {
    auto kern = pf_gemm_kernel<BN, SPLIT, Epi>;
    static bool attr_set = false;  // per instantiation
    if (!attr_set) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)PfTile<BN, SPLIT>::SMEM);
        if (e != cudaSuccess) return e;
        attr_set = true;
    }
    const dim3 grid((p.N + BN - 1) / BN, (p.M + PF_BM - 1) / PF_BM, zdim);
    kern<<<grid, PF_THREADS, PfTile<BN, SPLIT>::SMEM, m->stream>>>(a, a_lo, b, p, make_idesc(BN, bf16), epi);
    m->launches++;
    return cudaGetLastError();
}

// a: the activation's hi and lo maps (lo unused when split is off)
template <int BN, class Epi>
cudaError_t pf_launch(cd_model* m, bool split, const CUtensorMap (&a)[2], const CUtensorMap& b, const PfGemm& p, bool bf16, int zdim, const Epi& epi) {
    return split ? pf_launch_t<BN, true>(m, a[0], a[1], b, p, bf16, zdim, epi) : pf_launch_t<BN, false>(m, a[0], a[0], b, p, bf16, zdim, epi);
}

}  // namespace
}  // namespace cd
