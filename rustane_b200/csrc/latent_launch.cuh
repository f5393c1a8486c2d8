// One token of latent attention (the mla_* kernels of moe.cuh): absorbed queries and cache row, attention over the cached
// latents, merge and value projection.  Host side, shared by the families that have it.
#pragma once
#include "moe.cuh"
#include "step.cuh"

namespace {

struct MlaStep {
    MlaDims d;
    const float* qa;         // projections [heads (nope_n + rope_n) | latent_n | rope_n]
    const void *wuk_t, *wuv;  // [heads][latent][nope], [heads vdim][latent]
    const float* gamma;      // of the latent's norm
    Rotation rot;
    void* pool;              // the layer's pages
    float* qabs;             // [heads][latent + rope]
    void* qsplit;            // per block of 16 heads [2][16][latent + rope], zero where there is no head
    float *part_acc, *part_ml;  // [nsplit][heads][latent], [nsplit][heads][2]
    float* out;              // [heads vdim]
    int nsplit;
    float scale;
};

template <typename KT> bool mla_on_tensor_cores(const MlaDims& d) {
    return !std::is_same<KT, float>::value && d.latent % 16 == 0 && d.row() % 16 == 0 && mla_mma_smem_bytes(d.row()) <= (size_t)227 * 1024;
}

template <typename WT, typename KT>
cudaError_t launch_mla(cd_model* m, const MlaStep& p) {
    const MlaDims& d = p.d;
    cudaError_t e;
#define TRY(x) do { e = (x); if (e != cudaSuccess) return e; } while (0)
    const bool mma = mla_on_tensor_cores<KT>(d);
    TRY(launch_chain(m, mla_post_kernel<WT, KT>, dim3(mla_post_ctas(d)), dim3(128), mla_post_smem_floats(d) * sizeof(float), p.qa, (const WT*)p.wuk_t,
                     p.gamma, p.rot, (const int*)m->page_table, (const DevState*)m->st, (KT*)p.pool, p.qabs, mma ? (KT*)p.qsplit : (KT*)nullptr, d));
    if constexpr (!std::is_same<KT, float>::value) {
        if (mma) {
            const size_t smem = mla_mma_smem_bytes(d.row());
            auto go = [&](auto kern, int cols) {
                cudaError_t r = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
                if (r != cudaSuccess) return r;
                return launch_chain(m, kern, dim3(p.nsplit, d.head_blocks(), (d.latent + cols - 1) / cols), dim3(MLA_MMA_THREADS), smem, (const KT*)p.qsplit, (const KT*)p.pool,
                                    (const int*)m->page_table, (const DevState*)m->st, p.part_acc, p.part_ml, d, p.nsplit, p.scale, &m->st->error);
            };
            if (d.latent <= 128) TRY(go(mla_attn_mma_kernel<KT, 32>, 128));
            else if (d.latent <= 256) TRY(go(mla_attn_mma_kernel<KT, 64>, 256));
            else TRY(go(mla_attn_mma_kernel<KT, 128>, 512));
        }
    }
    if (!mma) {
        const size_t smem = mla_attn_smem_floats(d) * sizeof(float);
        TRY(cudaFuncSetAttribute(mla_attn_kernel<KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        TRY(launch_chain(m, mla_attn_kernel<KT>, dim3(p.nsplit, d.head_blocks(), d.col_blocks()), dim3(256), smem, (const float*)p.qabs, (const KT*)p.pool,
                         (const int*)m->page_table, (const DevState*)m->st, p.part_acc, p.part_ml, d, p.nsplit, p.scale));
    }
    return launch_chain(m, mla_out_kernel<WT>, dim3(d.heads, (d.vdim + 31) / 32), dim3(256), (d.latent + p.nsplit) * sizeof(float), (const float*)p.part_acc,
                        (const float*)p.part_ml, (const WT*)p.wuv, p.out, (const DevState*)m->st, d, p.nsplit, mma ? MLA_MMA_TILE : MLA_TILE);
#undef TRY
}

}  // namespace
