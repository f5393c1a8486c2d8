// What the step functions of all model families share: launching the streamed GEMV and the kernels of a
// token's chain, counting launches, the LM head and the head reductions / samplers that end a step.
#pragma once
#include <algorithm>
#include <string>
#include <type_traits>
#include <utility>

#include "kernels.cuh"
#include "model.h"

#define CK(m, call)                                                                              \
    do {                                                                                         \
        cudaError_t e_ = (call);                                                                 \
        if (e_ != cudaSuccess)                                                                   \
            return fail((m), CD_ERR_CUDA, std::string(#call) + ": " + cudaGetErrorString(e_));   \
    } while (0)

#define DISPATCH_WT(dtype, WT, ...)                                  \
    switch (dtype) {                                                 \
        case CD_DTYPE_F32: { typedef float WT; __VA_ARGS__; } break; \
        case CD_DTYPE_F16: { typedef __half WT; __VA_ARGS__; } break; \
        default: { typedef __nv_bfloat16 WT; __VA_ARGS__; } break;   \
    }
// storage of the embedding and the LM head (16-bit for the quantised kinds)
#define EMBED_DTYPE(m) (is_quant((m)->opt.weight_dtype) ? CD_DTYPE_BF16 : (m)->opt.weight_dtype)

namespace {
using namespace cd;

// kernel classes for per-class timing (cd_profile_decode_step)
enum { CLS_MISC = 0, CLS_QKV, CLS_ATTN, CLS_WO, CLS_W13, CLS_W2, CLS_HEAD, CLS_SAMPLE, CLS_COUNT };

inline size_t esize(int dtype) { return dtype == CD_DTYPE_F32 ? 4 : 2; }  // embedding, LM head, KV cache (never a quantised code)
inline bool is_quant(int dtype) { return dtype == CD_DTYPE_FP8_E4M3 || dtype == CD_DTYPE_INT4_G32; }
// bytes of one row of a linear with K inputs
inline size_t lin_row_bytes(int dtype, int K) {
    return dtype == CD_DTYPE_FP8_E4M3 ? Wfmt<Fp8Row>::row_stride(K) : dtype == CD_DTYPE_INT4_G32 ? Wfmt<Int4G32>::row_stride(K) : (size_t)K * esize(dtype);
}
inline size_t align_up(size_t v, size_t a) { return (v + a - 1) / a * a; }

// ------------------------------------------------------------------ GEMV launch
template <typename WT, int NITER, int R, int UNIT, bool NORM, class Epi, class Src = SrcPlain, class In = GemvIn>
cudaError_t gemv_go(cd_model* m, const WT* W, const float* x, const float* gamma, float* norm_out, int N, int K,
                    int NT, const Epi& epi, const Src& src_in = Src{}, const In& in = In{}) {
    Src src = src_in;
    int nunits_all = N / UNIT, K1 = K;  // K1: the widest row
    if constexpr (Src::PAIR) {
        nunits_all += src.n2 / UNIT;
        K1 = std::max(K, src.k2);
    }
    {
        // one persistent CTA per SM, ring of up to eight 16-24 KB stages
        constexpr int G = Wfmt<WT>::QUANT ? 2 : 1;  // consumer groups: the quantised formats need twice the decode warps
        constexpr int RT = G == 2 ? (NITER == 1 ? 8 : 4) : NITER == 1 ? 4 : NITER == 2 ? 2 : 1;
        auto tk = gemv_tma_kernel<WT, NITER, RT, UNIT, NORM, Epi, G, Src, In>;
        const int grid = std::max(1, std::min(nunits_all, m->sm_count));
        int rows_cap = (nunits_all / grid + 1) * UNIT;
        if constexpr (Src::PAIR) {
            if (grid < 2) return cudaErrorInvalidConfiguration;
            const double b1 = (double)(N / UNIT) * K, b2 = (double)(src.n2 / UNIT) * src.k2;
            src.split = std::max(1, std::min(grid - 1, (int)(grid * b1 / (b1 + b2) + 0.5)));
            rows_cap = std::max(N / UNIT / src.split + 1, src.n2 / UNIT / (grid - src.split) + 1) * UNIT;
        }
        const size_t stage_bytes = (size_t)RT * Wfmt<WT>::row_stride(K1);
        const size_t fixed = ((size_t)rows_cap * (GEMV_CONSUMERS / 32) + 32) * sizeof(float) + 2 * 8 * 8 + 128;
        const size_t budget = (size_t)m->ring_kb * 1024;
        const int nstages = fixed + 2 * stage_bytes <= budget ? (int)std::min<size_t>(8, (budget - fixed) / stage_bytes) : 0;
        if (nstages >= 2) {
            // never less than half an SM's shared memory: two of these CTAs (of consecutive kernels, under programmatic
            // dependent launch) on one SM measured 16 % slower per token and, rarely, gave run-to-run different logits
            const size_t smem = std::max((size_t)nstages * stage_bytes + fixed, (size_t)116 * 1024);
            static size_t smem_set = 0;  // per instantiation
            if (smem > smem_set) {
                cudaError_t e = cudaFuncSetAttribute(tk, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
                if (e != cudaSuccess) return e;
                smem_set = smem;
            }
            cudaLaunchConfig_t lc = {};
            lc.gridDim = dim3(grid);
            lc.blockDim = dim3(G * GEMV_CONSUMERS + 32);
            lc.dynamicSmemBytes = smem;
            lc.stream = m->stream;
            cudaLaunchAttribute at[1];
            at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
            at[0].val.programmaticStreamSerializationAllowed = 1;
            lc.attrs = at;
            lc.numAttrs = m->pdl ? 1 : 0;
            NextStream next = m->next_stream;
            next.test_drop = (m->opt.test_flags & 8) ? 1 : 0;
            if (next.w && std::min(next.nunits, m->sm_count) != grid) next.w = nullptr;  // partitions would not line up
            m->next_stream.w = nullptr;
            TpLink tp = m->tp;
            tp.in_reduce = m->tp_in.in_reduce; tp.res = m->tp_in.res; tp.alpha = m->alpha; tp.x_out = m->tp_in.x_out; tp.ar_out = 0;
            m->tp_in.in_reduce = 0;
            cudaError_t e = cudaLaunchKernelEx(&lc, tk, W, x, gamma, norm_out, N, K, rows_cap, nstages, &m->st->error, next, tp, epi, src, m->rms_eps, in);
            count_launch(m);
            return e;
        }
    }
    return cudaErrorInvalidConfiguration;  // a stage of this shape does not fit the ring twice
}

// N and K of a gathered source (Src::DYNAMIC) are the upper bounds of its shape.  cudaErrorInvalidValue: no
// instantiation takes a K this wide (the caller may have another kernel for it).
template <typename WT, int UNIT, bool NORM, class Epi, class Src = SrcPlain, class In = GemvIn>
cudaError_t launch_gemv(cd_model* m, const void* W, const float* x, const float* gamma, float* norm_out, int N, int K,
                        const Epi& epi, const Src& src = Src{}, const In& in = In{}) {
    constexpr int EPC = Wfmt<WT>::EPC;
    int nchunks = K / EPC;
    if constexpr (Src::PAIR) nchunks = std::max(K, src.k2) / EPC;
    const int NT = std::min(256, (nchunks + 31) / 32 * 32);
    const int niter = (nchunks + NT - 1) / NT;
    const WT* w = reinterpret_cast<const WT*>(W);
    switch (niter) {
        case 1: return gemv_go<WT, 1, 8, UNIT, NORM, Epi, Src, In>(m, w, x, gamma, norm_out, N, K, NT, epi, src, in);
        case 2: return gemv_go<WT, 2, 4, UNIT, NORM, Epi, Src, In>(m, w, x, gamma, norm_out, N, K, NT, epi, src, in);
        case 3: return gemv_go<WT, 3, 2, UNIT, NORM, Epi, Src, In>(m, w, x, gamma, norm_out, N, K, NT, epi, src, in);
        case 4: return gemv_go<WT, 4, 2, UNIT, NORM, Epi, Src, In>(m, w, x, gamma, norm_out, N, K, NT, epi, src, in);
        default: break;
    }
    if constexpr (!Wfmt<WT>::QUANT) {  // the quantised formats hold 16 / 32 elements of x per chunk: four chunks per thread at most
        switch (niter) {
            case 5:
            case 6: return gemv_go<WT, 6, 2, UNIT, NORM, Epi, Src, In>(m, w, x, gamma, norm_out, N, K, NT, epi, src, in);
            case 7:
            case 8: return gemv_go<WT, 8, 1, UNIT, NORM, Epi, Src, In>(m, w, x, gamma, norm_out, N, K, NT, epi, src, in);
            default: break;
        }
    }
    return cudaErrorInvalidValue;
}

// What follows the layers: nothing (hidden state wanted), or the final RMSNorm + LM head and the head reduction /
// sampler the step asks for.  `ars`: all-reduces the token issued (tensor / expert parallel), `last_ar`: index of the
// one whose sum is still in the inboxes.  WT: storage of the LM head; LT: row format of the next token's first GEMV; HeadIn:
// how the head's input comes about where that is not RMSNorm of x_a (an input type of the streamed GEMV, kernels.cuh).
template <typename WT, typename LT, class HeadIn = GemvIn>
cudaError_t enqueue_head_t(cd_model* m, const cd_step& p, bool use_mega, unsigned int ars, int last_ar, const HeadIn& head_in = HeadIn{}) {
    const cd_config& c = m->cfg;
    cudaError_t e;
#define TRY(x) do { e = (x); if (e != cudaSuccess) return e; } while (0)
    // a vocabulary-sharded head exchanges candidates between the ranks; under expert parallelism the head is replicated
    const bool xhead = m->tp_world > 1 && !m->replicated_head;
    const TpLink htp = xhead ? m->tp : TpLink{};
    m->cur_cls = CLS_MISC;
    if (p.head == HEAD_NONE) {
        if (m->tp_world > 1) {  // nobody else reads the last all-reduce of this token: consume it
            TpLink tp = m->tp;
            tp.in_reduce = last_ar; tp.res = m->x_b; tp.x_out = m->x_a; tp.alpha = m->alpha;
            tp_consume_kernel<<<8, 256, 0, m->stream>>>(tp, &m->st->error);
            count_launch(m);
        }
        advance_kernel<<<1, 1, 0, m->stream>>>(m->st, ars);
        count_launch(m);
        return cudaGetLastError();
    }
    // encode_rmsnorm(gamma_final) + LM head (lib.rs:867-986), logits left in HBM
    m->cur_cls = CLS_HEAD;
    if (!use_mega) {
    m->next_stream = NextStream{m->prefetch_kb > 0 ? m->layers[0].wqkv : nullptr, Wfmt<LT>::row_stride(c.dim),
                                (c.q_dim + 2 * c.kv_dim) / 2, 2, (uint32_t)m->prefetch_kb * 1024u};
    if (m->tp_world > 1) { m->tp_in.in_reduce = last_ar; m->tp_in.res = m->x_b; m->tp_in.x_out = m->x_a; }
    if constexpr (HeadIn::CUSTOM) TRY((launch_gemv<WT, 1, false>(m, m->lm_head, m->x_a, nullptr, nullptr, m->v_loc, c.dim, EpiStore{m->logits}, SrcPlain{}, head_in)));
    else TRY((launch_gemv<WT, 1, true>(m, m->lm_head, m->x_a, m->gamma_final, m->norm_final, m->v_loc, c.dim, EpiStore{m->logits})));
    }
    unsigned int* head_counter = m->counters + c.heads;
    m->cur_cls = CLS_SAMPLE;
    bool count_ars = m->tp_world > 1 && !xhead;  // the single-GPU head kernels do not count the token's all-reduces
    switch (p.head) {
        case HEAD_LOGITS:
            advance_kernel<<<1, 1, 0, m->stream>>>(m->st, ars);
            count_ars = false;
            break;
        case HEAD_ARGMAX:
        case LOOP_GREEDY:
            head_argmax_kernel<<<m->nblocks, 256, 0, m->stream>>>(m->logits, m->v_loc, m->block_vals, m->block_idxs, head_counter,
                                                                 m->out_token, m->st, m->out_ring, p.head == LOOP_GREEDY, m->v0, htp);
            if (xhead) {
                count_launch(m);
                tp_pick_kernel<<<1, 32, 0, m->stream>>>(m->tp, m->out_token, m->st, m->out_ring, p.head == LOOP_GREEDY, ars);
            }
            break;
        case HEAD_TOPK:
        case LOOP_TOPK:
            head_topk_kernel<<<m->nblocks, 256, 0, m->stream>>>(m->logits, m->v_loc, p.k, m->topk_vals, m->topk_idxs);
            count_launch(m);
            if (p.head == LOOP_TOPK && xhead) {
                // every rank's candidates to every rank, then the same merge and draw everywhere
                tp_push_topk_kernel<<<1, 256, 0, m->stream>>>(m->tp, m->topk_vals, m->topk_idxs, m->nblocks, m->tp_nb, p.k, m->v0);
                tp_wait_topk_kernel<<<1, 256, 0, m->stream>>>(m->tp, m->st, m->tp_topk_vals, m->tp_topk_idxs, m->tp_nb, m->tp_nb * 32);
                sample_topk_kernel<<<1, 1024, 0, m->stream>>>(m->tp_topk_vals, m->tp_topk_idxs, m->tp_world * m->tp_nb * 32, p.k, p.t, p.softcap,
                                                              m->st, m->out_ring);
                count_launch(m); count_launch(m); count_launch(m);
                tp_count_allreduces_kernel<<<1, 1, 0, m->stream>>>(m->st, ars);
            } else if (p.head == LOOP_TOPK)
                sample_topk_kernel<<<1, 1024, 0, m->stream>>>(m->topk_vals, m->topk_idxs, m->nblocks * p.k, p.k, p.t, p.softcap,
                                                              m->st, m->out_ring);
            else {
                if (xhead) {  // the per-token call: every rank's candidates to every rank, the host copies them out in block order
                    tp_push_topk_kernel<<<1, 256, 0, m->stream>>>(m->tp, m->topk_vals, m->topk_idxs, m->nblocks, m->tp_nb, p.k, m->v0);
                    tp_wait_topk_kernel<<<1, 256, 0, m->stream>>>(m->tp, m->st, m->tp_topk_vals, m->tp_topk_idxs, m->tp_nb, m->tp_nb * 32);
                    count_launch(m); count_launch(m);
                }
                advance_kernel<<<1, 1, 0, m->stream>>>(m->st, ars);
                count_ars = false;
            }
            break;
        case HEAD_STATS:
        case LOOP_FULLVOCAB:
            head_stats_kernel<<<m->nblocks, 256, 0, m->stream>>>(m->logits, m->v_loc, p.inv_t, p.softcap, m->maxes, m->sums);
            count_launch(m);
            if (p.head == LOOP_FULLVOCAB && xhead) {
                // every rank's per-block (max, sum) to every rank; all pick the same block, its owner draws the token
                tp_push_topk_kernel<<<1, 256, 0, m->stream>>>(m->tp, m->maxes, reinterpret_cast<const uint32_t*>(m->sums), m->nblocks, m->tp_nb, 1, 0);
                tp_wait_topk_kernel<<<1, 256, 0, m->stream>>>(m->tp, m->st, m->tp_topk_vals, m->tp_topk_idxs, m->tp_nb, m->tp_nb);
                count_launch(m); count_launch(m);
                tp_sample_fullvocab_kernel<<<1, 256, 0, m->stream>>>(m->logits, m->v0, m->full_cfg.vocab, m->tp_topk_vals, m->tp_topk_idxs, m->tp_nb,
                                                                    p.t, p.softcap, m->st, m->out_ring, m->tp, ars);
            } else if (p.head == LOOP_FULLVOCAB)
                sample_fullvocab_kernel<<<1, 256, 0, m->stream>>>(m->logits, c.vocab, m->maxes, m->sums, m->nblocks, p.t, p.softcap,
                                                                 m->st, m->out_ring);
            else {
                advance_kernel<<<1, 1, 0, m->stream>>>(m->st, ars);
                count_ars = false;
            }
            break;
        default: return cudaErrorInvalidValue;
    }
    count_launch(m);
    if (count_ars) {
        tp_count_allreduces_kernel<<<1, 1, 0, m->stream>>>(m->st, ars);
        count_launch(m);
    }
    return cudaGetLastError();
#undef TRY
}

// A launch in the token's chain of kernels: under programmatic dependent launch the kernel may become resident while
// its predecessor still runs (each of them waits, griddepcontrol.wait, before it touches anything the chain produced).
template <typename... KArgs, typename... Args>
cudaError_t launch_chain(cd_model* m, void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, Args&&... args) {
    cudaLaunchConfig_t lc = {};
    lc.gridDim = grid;
    lc.blockDim = block;
    lc.dynamicSmemBytes = smem;
    lc.stream = m->stream;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = 1;
    lc.attrs = at;
    lc.numAttrs = m->pdl ? 1 : 0;
    const cudaError_t e = cudaLaunchKernelEx(&lc, kern, std::forward<Args>(args)...);
    count_launch(m);
    return e;
}

// final norm + LM head on the hidden state in x_a; logits stay in HBM, the state is not advanced
template <typename WT>
cudaError_t enqueue_head_only_t(cd_model* m) {
    m->cur_cls = CLS_HEAD;
    m->next_stream.w = nullptr;
    return launch_gemv<WT, 1, true>(m, m->lm_head, m->x_a, m->gamma_final, m->norm_final, m->v_loc, m->cfg.dim, EpiStore{m->logits});
}

}  // namespace
