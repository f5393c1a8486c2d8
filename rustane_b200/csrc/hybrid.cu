// The configured decoder family (hybrid.h): construction from a model folder (config.json + model.safetensors) or from a
// configuration with synthetic weights, the per-token step, and the recurrent state's snapshots.
//
// A step, per layer run (each line a kernel of the token's chain, programmatic dependent launch between them):
//   gemv_tma_kernel     every projection of the mixer's input; its prologue forms the residual stream behind the
//                       previous sublayer and the norm ahead of this one (InResidual / InParallelMix)
//   mixer_step_kernel   the mixers, cache append, state update; latent attention: mla_post / mla_attn / mla_out
//   gemv_tma_kernel     the output projection, a linear attention's norm and gate in its prologue (InGatedNorm); of two
//                       parallel mixers both in one launch (SrcPair, InMixerOutputs)
//   gemv_tma_kernel     gate | up with the norms and residual in its prologue; for a mixture of experts
//                       moe_router_kernel does that and the chosen experts' rows are gathered (SrcExpertRows)
//   gemv_tma_kernel     down (SrcExpertCols)
//   gemv_tma_kernel     token side, where the model has it: gate, times the token's part of the second embedding (EpiTokenGate)
//   gemv_tma_kernel     its projection back to the width
#include <algorithm>
#include <cmath>
#include <cstring>
#include <fstream>
#include <iterator>
#include <memory>

#include "step.cuh"
#include "latent_launch.cuh"
#include "mixers.cuh"
#include "hybrid.h"
#include "safetensors.h"

using namespace cd;

namespace {

// ------------------------------------------------------------------ the step
template <typename WT, typename KT>
cudaError_t hybrid_step_t(cd_model* m, const cd_step& p) {
    const cd_config& c = m->cfg;
    cd_hybrid_state& S = *m->hybrid;
    const float mult = S.cfg.residual_mult, eps = S.cfg.eps;
    const int D = c.dim, n = S.cfg.width;  // width padded to 8 with zeros, and the model's own
    cudaError_t e;
#define TRY(x) do { e = (x); if (e != cudaSuccess) return e; } while (0)
    m->cur_cls = CLS_MISC;
    m->next_stream.w = nullptr;
    if (p.input == 2) {
        next_prompt_kernel<<<1, 1, 0, m->stream>>>(m->st, m->prompt_dev);
        count_launch(m);
    }
    if (p.input >= 1) {
        embed_kernel<WT><<<std::max(1, D / 256), 256, 0, m->stream>>>((const WT*)m->embed, m->st, m->x_a, D, m->full_cfg.vocab);
        count_launch(m);
        TRY(cudaGetLastError());
    }
    float* x[2] = {m->x_a, m->x_b};  // the residual stream alternates: a kernel that forms the next one reads the last one
    int cur = 0;
    // the last sublayer's output, still to be normed and added: y, or two parallel mixers' outputs of layer `pair`
    struct { const float* y; VecNorm post; const cd_hybrid_layer* pair; } behind = {nullptr, {}, nullptr};
    float *yl = S.y, *yr = S.y + D;
    auto residual = [&](const VecNorm& pre, const float* add = nullptr) { return InResidual{x[cur], behind.y, add, x[cur ^ 1], behind.post, pre, mult, eps, n}; };
    auto mix_in = [&](const cd_hybrid_layer& L) { return InParallelMix{x[cur], yl, yr, L.out_l, L.out_r, L.post1.w, x[cur ^ 1], mult, eps, n}; };
    // the next GEMV's first rows, pulled into L2 behind a GEMV's own last loads
    auto hint = [&](const void* w, int K, int N, int unit) {
        m->next_stream = NextStream{m->prefetch_kb > 0 ? w : nullptr, Wfmt<WT>::row_stride(K), N / unit, unit, (uint32_t)m->prefetch_kb * 1024u};
    };
    const int nruns = (int)S.runs.size(), side = S.cfg.side_dim;
    for (int r = 0; r < nruns; ++r) {
        const cd_hybrid_layer& L = S.layers[S.runs[r].layer];
        const cd_hybrid_layer* next = r + 1 < nruns ? &S.layers[S.runs[r + 1].layer] : nullptr;
        auto hint_next = [&]() {  // what follows the layer's last sublayer
            if (side) hint(L.side_gate, D, side, 1);
            else if (next) hint(next->wmix, D, next->proj.rows, 1);
            else if (p.head != HEAD_NONE) hint(m->lm_head, D, m->v_loc, 1);
        };
        m->cur_cls = CLS_QKV;
        const EpiStore to_proj{S.proj};
        if (behind.pair) TRY((launch_gemv<WT, 1, false>(m, L.wmix, x[cur], nullptr, nullptr, L.proj.rows, D, to_proj, SrcPlain{}, mix_in(*behind.pair))));
        else TRY((launch_gemv<WT, 1, false>(m, L.wmix, x[cur], nullptr, nullptr, L.proj.rows, D, to_proj, SrcPlain{}, residual(L.pre1, S.step_vector(S.runs[r])))));
        cur ^= 1;
        m->cur_cls = CLS_ATTN;
        void* kv = m->layers[r].kv;
        if (L.cfg.mixer == HybridLayerCfg::LATENT) {
            TRY((launch_mla<WT, KT>(m, MlaStep{L.ld, S.proj, L.wuk_t, L.wuv, L.latent_norm, Rotation{nullptr, L.freq, L.ld.rot_dims}, kv, S.qabs, S.qsplit, S.part_acc, S.part_ml,
                                               S.attn, L.nsplit, L.cfg.latent.scale})));
        } else {
            MixerStep q;
            q.a = L.ad; q.d = L.md; q.pl = L.proj; q.proj = S.proj;
            q.q_norm = L.q_norm; q.k_norm = L.k_norm; q.sink = L.sink; q.slopes = L.slopes; q.ib = L.ib; q.fb = L.fb;
            q.page_table = m->page_table; q.st = m->st;
            q.part_acc = S.part_acc; q.part_ml = S.part_ml; q.counters = S.counters;
            q.attn = S.attn; q.mem = S.mem; q.ssq = S.ssq; q.state = S.state + S.state_off[r]; q.nsplit = L.nsplit;
            const size_t smem = std::max(mixer_attn_smem_floats(L.ad.kr(), L.ad.vp, L.ad.maps), mixer_mem_smem_floats(L.md.dim)) * sizeof(float);
            auto go = [&](auto kern) {
                if (smem > 48 * 1024) {
                    const cudaError_t r_ = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
                    if (r_ != cudaSuccess) return r_;
                }
                return launch_chain(m, kern, dim3(L.md.H * L.md.nslice + L.ad.H * L.nsplit), dim3(MIX_THREADS), smem, q, (KT*)kv);
            };
            if (L.ad.maps == 2) TRY(go(mixer_step_kernel<KT, 2>));
            else TRY(go(mixer_step_kernel<KT, 1>));
        }
        m->cur_cls = CLS_WO;
        const FfnCfg& f = L.cfg.mlp;
        if (f.kind == FfnCfg::DENSE) hint(L.w13, D, 2 * L.ffp, 2);
        else if (f.kind == FfnCfg::NONE) hint_next();
        behind = {S.y, L.post1, nullptr};
        if (L.cfg.mixer == HybridLayerCfg::PARALLEL) {
            const InMixerOutputs in{S.attn, S.mem, S.ssq, L.mem_norm, S.proj + L.proj.rg, L.md.H * L.md.vdim, L.md.vdim, L.md.nslice, eps};
            TRY((launch_gemv<WT, 1, false>(m, L.wo_l, S.attn, nullptr, nullptr, D, L.kl, EpiStore{S.y}, SrcPair{L.wo_r, D, L.kr, 0}, in)));
            behind.pair = &L;
        } else if (L.cfg.mixer == HybridLayerCfg::MEMORY) {
            const InGatedNorm in{S.mem, L.mem_norm, S.proj + L.proj.rg, L.md.H * L.md.vdim, eps};
            TRY((launch_gemv<WT, 1, false>(m, L.wo_l, S.mem, nullptr, nullptr, D, L.kl, EpiStore{S.y}, SrcPlain{}, in)));
        } else {
            TRY((launch_gemv<WT, 1, false>(m, L.wo_l, S.attn, nullptr, nullptr, D, L.kl, EpiStore{S.y})));
        }
        if (f.kind == FfnCfg::DENSE) {
            m->cur_cls = CLS_W13;
            hint(L.w2, L.ffp, D, 1);
            const EpiGate to_gate{S.gate, CD_ACT_SWIGLU};
            if (behind.pair) TRY((launch_gemv<WT, 2, false>(m, L.w13, x[cur], nullptr, nullptr, 2 * L.ffp, D, to_gate, SrcPlain{}, mix_in(L))));
            else TRY((launch_gemv<WT, 2, false>(m, L.w13, x[cur], nullptr, nullptr, 2 * L.ffp, D, to_gate, SrcPlain{}, residual(L.pre2))));
            cur ^= 1;
            m->cur_cls = CLS_W2;
            hint_next();
            TRY((launch_gemv<WT, 1, false>(m, L.w2, S.gate, nullptr, nullptr, D, L.ffp, EpiStore{S.y2})));
        } else if (f.kind == FfnCfg::MOE) {  // behind two parallel mixers
            m->cur_cls = CLS_W13;
            int* sel = S.sel_ids + (size_t)S.runs[r].layer * SRC_MAX_LIST;
            TRY(launch_chain(m, moe_router_kernel<WT, RouterMixIn>, dim3((f.experts + 3) / 4), dim3(128), (size_t)std::max(D, f.experts + f.groups) * sizeof(float),
                             RouterMixIn{x[cur], yl, yr, L.out_l, L.out_r, L.post1.w, x[cur ^ 1], mult, eps, n}, (const WT*)L.wr, S.router_logits, S.router_counter, sel,
                             S.sel_w, S.loc_ids, S.loc_w, S.n_loc, D, RouteRule{f.experts, f.top, f.groups, f.keep}, 0, f.experts));
            cur ^= 1;
            const int units = f.top * L.ffp;
            const uint32_t es = (uint32_t)sizeof(WT);
            if (L.stream_ffn) {
                const SrcExpertRows s13{S.loc_ids, S.n_loc, nullptr, 2 * L.ffp, 0};
                TRY((launch_gemv<WT, 2, false>(m, L.w13, x[cur], nullptr, nullptr, 2 * units, D, EpiGateMoe{S.gate, S.loc_w, S.n_loc, L.ffp}, s13)));
                m->cur_cls = CLS_W2;
                hint_next();
                const SrcExpertCols s2{S.loc_ids, S.n_loc, nullptr, L.ffp, 0, D, (uint32_t)L.ffp * es, 0};
                TRY((launch_gemv<WT, 1, false>(m, L.w2, S.gate, nullptr, nullptr, D, units, EpiStore{S.y2}, s2)));
            } else {
                const MoePick pick{S.loc_ids, S.loc_w, S.n_loc};
                const MoeDims ed{D, L.ffp, 0};
                TRY(launch_chain(m, moe_w13_kernel<WT>, dim3((units + 7) / 8), dim3(256), D * sizeof(float), (const float*)x[cur], (const WT*)L.w13, (const WT*)nullptr, pick,
                                 S.gate, ed));
                m->cur_cls = CLS_W2;
                TRY(launch_chain(m, moe_w2_kernel<WT>, dim3((D + 7) / 8), dim3(256), units * sizeof(float), (const float*)S.gate, (const WT*)L.w2, (const WT*)nullptr, pick,
                                 (const float*)S.zero, S.y2, 1.0f, ed, TpLink{}));
            }
        }
        if (f.kind != FfnCfg::NONE) behind = {S.y2, L.post2, nullptr};
        if (side) {
            m->cur_cls = CLS_MISC;
            hint(L.side_proj, S.side_pad(), D, 1);
            const EpiTokenGate<WT> to_side{S.side, (const WT*)S.side_embed + (size_t)S.runs[r].layer * side, S.side_ld(), m->full_cfg.vocab, m->st};
            TRY((launch_gemv<WT, 1, false>(m, L.side_gate, x[cur], nullptr, nullptr, side, D, to_side, SrcPlain{}, residual(VecNorm{}))));
            cur ^= 1;
            if (next) hint(next->wmix, D, next->proj.rows, 1);
            else if (p.head != HEAD_NONE) hint(m->lm_head, D, m->v_loc, 1);
            TRY((launch_gemv<WT, 1, false>(m, L.side_proj, S.side, nullptr, nullptr, D, S.side_pad(), EpiStore{S.y})));
            behind = {S.y, L.side_norm, nullptr};
        }
    }
    m->cur_cls = CLS_MISC;
    if (behind.pair) {
        InParallelMix in = mix_in(*behind.pair);
        in.x_out = m->x_a;
        TRY(launch_chain(m, vector_input_kernel<InParallelMix>, dim3(1), dim3(GEMV_CONSUMERS), 0, in, D));
        const InResidual head_in{m->x_a, nullptr, nullptr, m->x_b, VecNorm{}, S.final_norm, mult, eps, n};
        return enqueue_head_t<WT, WT, InResidual>(m, p, false, 0u, 0, head_in);
    }
    if (p.head == HEAD_NONE) {
        InResidual in = residual(VecNorm{});
        in.x_out = m->x_a;
        TRY(launch_chain(m, vector_input_kernel<InResidual>, dim3(1), dim3(GEMV_CONSUMERS), 0, in, D));
        return enqueue_head_t<WT, WT>(m, p, false, 0u, 0);
    }
    return enqueue_head_t<WT, WT, InResidual>(m, p, false, 0u, 0, residual(S.final_norm));
#undef TRY
}

cudaError_t hybrid_step(cd_model* m, const cd_step& p) {
    if (m->opt.weight_dtype == CD_DTYPE_F32) return hybrid_step_t<float, float>(m, p);
    return m->kv_dtype == CD_DTYPE_F16 ? hybrid_step_t<__nv_bfloat16, __half>(m, p) : hybrid_step_t<__nv_bfloat16, __nv_bfloat16>(m, p);
}

// final norm and LM head on the hidden state in x_a
template <typename WT> cudaError_t hybrid_head_only_t(cd_model* m) {
    const cd_hybrid_state& S = *m->hybrid;
    m->cur_cls = CLS_HEAD;
    m->next_stream.w = nullptr;
    const InResidual in{m->x_a, nullptr, nullptr, m->x_b, VecNorm{}, S.final_norm, 1.0f, S.cfg.eps, S.cfg.width};
    return launch_gemv<WT, 1, false>(m, m->lm_head, m->x_a, nullptr, nullptr, m->v_loc, m->cfg.dim, EpiStore{m->logits}, SrcPlain{}, in);
}
cudaError_t hybrid_head_only(cd_model* m) { return m->opt.weight_dtype == CD_DTYPE_F32 ? hybrid_head_only_t<float>(m) : hybrid_head_only_t<__nv_bfloat16>(m); }

// ------------------------------------------------------------------ recurrent state: snapshots at earlier lengths
float* slot_ptr(const cd_hybrid_state& S, int i) { return S.state + (size_t)i * S.slot_floats; }

int find_slot(const cd_hybrid_state& S, size_t len) {
    for (int i = 1; i < cd_hybrid_state::SLOTS; ++i)
        if (S.slot_len[i] == len) return i;
    return 0;
}

int hybrid_mark(cd_model* m) {
    cd_hybrid_state& S = *m->hybrid;
    int s = find_slot(S, m->len);
    for (int i = 1; !s && i < cd_hybrid_state::SLOTS; ++i)
        if (S.slot_len[i] == cd_hybrid_state::FREE) s = i;
    if (!s) {  // the one that was not used for longest
        s = 1;
        for (int i = 2; i < cd_hybrid_state::SLOTS; ++i)
            if (S.slot_used[i] < S.slot_used[s]) s = i;
    }
    CK(m, cudaMemcpyAsync(slot_ptr(S, s), S.state, S.slot_floats * 4, cudaMemcpyDeviceToDevice, m->stream));
    S.slot_len[s] = m->len;
    S.slot_used[s] = ++S.clock;
    return CD_OK;
}

bool hybrid_can_rewind(const cd_model* m, size_t len) {
    return len == 0 || (len == m->len && m->state_len == len) || find_slot(*m->hybrid, len) > 0;
}

int hybrid_rewind(cd_model* m, size_t len) {
    cd_hybrid_state& S = *m->hybrid;
    if (!(len == m->len && m->state_len == len)) {
        if (len == 0) {
            CK(m, cudaMemsetAsync(S.state, 0, S.slot_floats * 4, m->stream));
        } else {
            const int s = find_slot(S, len);
            if (!s) return fail(m, CD_ERR_UNSUPPORTED, "the recurrent state at length " + std::to_string(len) + " is not kept (it is at the ends of the last prompt passes)");
            CK(m, cudaMemcpyAsync(S.state, slot_ptr(S, s), S.slot_floats * 4, cudaMemcpyDeviceToDevice, m->stream));
            S.slot_used[s] = ++S.clock;
        }
    }
    for (int i = 1; i < cd_hybrid_state::SLOTS; ++i)  // what follows may differ from what was there
        if (S.slot_len[i] != cd_hybrid_state::FREE && S.slot_len[i] > len) S.slot_len[i] = cd_hybrid_state::FREE;
    m->state_len = len;
    return CD_OK;
}

void hybrid_release(cd_model* m) {
    if (!m->hybrid) return;
    hybrid_prefill_release(m);
    if (m->hybrid->ws) cudaFree(m->hybrid->ws);
    if (m->hybrid->state) cudaFree(m->hybrid->state);
    delete m->hybrid;
    m->hybrid = nullptr;
}

const cd_family HYBRID_FAMILY = {"hybrid", hybrid_step, hybrid_head_only, hybrid_prefill, hybrid_hidden_row, nullptr, hybrid_release, hybrid_mark, hybrid_can_rewind, hybrid_rewind};

// ------------------------------------------------------------------ weights
// a head's block of rows transposed: src [heads * block][in] -> dst [heads][ld_rows][ld], dst row (h, c), column d = src row
// (h block + d), column c; zeros elsewhere (the arena starts out zero)
template <typename WT>
__global__ void transpose_heads_kernel(const WT* __restrict__ src, WT* __restrict__ dst, int heads, int block, int in, int src_ld, int ld_rows, int ld) {
    const size_t total = (size_t)heads * block * in;
    for (size_t j = (size_t)blockIdx.x * blockDim.x + threadIdx.x; j < total; j += (size_t)gridDim.x * blockDim.x) {
        const size_t d = j % block, c = j / block % in, h = j / block / in;
        dst[(h * ld_rows + c) * ld + d] = src[(h * block + d) * src_ld + c];
    }
}
// dst[(o * row_mul + row_off) * ld + i] = src[o * in + i], columns in .. ld - 1 zero.  src_kind 0: bf16, 1: f16, 2: f32.
template <typename WT>
__global__ void place_rows_kernel(const void* __restrict__ src, int src_kind, WT* __restrict__ dst, int in, int out, int ld, int row_mul, int row_off) {
    const size_t total = (size_t)out * ld;
    for (size_t j = (size_t)blockIdx.x * blockDim.x + threadIdx.x; j < total; j += (size_t)gridDim.x * blockDim.x) {
        const size_t o = j / ld, i = j % ld, at = o * in + i;
        float v = 0.0f;
        if (i < (size_t)in)
            v = src_kind == 0 ? __bfloat162float(((const __nv_bfloat16*)src)[at]) : src_kind == 1 ? __half2float(((const __half*)src)[at]) : ((const float*)src)[at];
        dst[(o * row_mul + row_off) * ld + i] = Elem<WT>::from_f32(v);
    }
}
template <typename WT>
__global__ void synth_rows_kernel(WT* __restrict__ dst, int in, int out, int ld, int row_mul, int row_off, uint64_t key, float scale) {
    const size_t total = (size_t)out * ld;
    for (size_t j = (size_t)blockIdx.x * blockDim.x + threadIdx.x; j < total; j += (size_t)gridDim.x * blockDim.x) {
        const size_t o = j / ld, i = j % ld;
        dst[(o * row_mul + row_off) * ld + i] = Elem<WT>::from_f32(i < (size_t)in ? synth_value(key, o * in + i, scale) : 0.0f);
    }
}

// Where tensors come from: a safetensors file, or the counter-based generator (keyed by the tensor's name).
struct TensorSource {
    const SafeTensors* file = nullptr;
    uint64_t seed = 0;
    float std = 0.02f;
    cd_model* m = nullptr;
    int rc = CD_OK;

    uint64_t key(const std::string& name) const {
        uint64_t h = 1469598103934665603ull;  // FNV-1a of the name
        for (unsigned char ch : name) h = (h ^ ch) * 1099511628211ull;
        return synth_key(seed, h);
    }
    const TensorView* need(const std::string& name, std::vector<size_t> shape) {
        const TensorView* t = file->find(name);
        if (!t) { rc = fail(m, CD_ERR_IO, "missing tensor " + name); return nullptr; }
        if (t->shape != shape) { rc = fail(m, CD_ERR_IO, "tensor " + name + " does not have the shape the configuration implies"); return nullptr; }
        if (t->dtype != "BF16" && t->dtype != "F16" && t->dtype != "F32") { rc = fail(m, CD_ERR_IO, "tensor " + name + " has unsupported type " + t->dtype); return nullptr; }
        return t;
    }
    // a matrix [out, in] into rows of `ld` elements
    void matrix(const std::string& name, void* dst, int out, int in, int ld, int row_mul = 1, int row_off = 0) {
        if (rc) return;
        const size_t total = (size_t)out * ld;
        const int grid = (int)std::min<size_t>((size_t)m->sm_count * 8, (total + 255) / 256);
        const bool f32 = m->opt.weight_dtype == CD_DTYPE_F32;
        cudaError_t e;
        if (file) {
            const TensorView* t = need(name, {(size_t)out, (size_t)in});
            if (!t) return;
            if (m->staging_bytes < t->bytes) {
                if (m->staging) cudaFree(m->staging);
                m->staging = nullptr;
                m->staging_bytes = 0;
                e = cudaMalloc(&m->staging, t->bytes);
                if (e != cudaSuccess) { rc = fail(m, CD_ERR_CUDA, std::string("weight staging: ") + cudaGetErrorString(e)); return; }
                m->staging_bytes = t->bytes;
            }
            e = cudaMemcpyAsync(m->staging, t->data, t->bytes, cudaMemcpyHostToDevice, m->stream);  // (stream order: the last tensor was placed before)
            const int kind = t->dtype == "BF16" ? 0 : t->dtype == "F16" ? 1 : 2;
            if (e == cudaSuccess) {
                if (f32) place_rows_kernel<float><<<grid, 256, 0, m->stream>>>(m->staging, kind, (float*)dst, in, out, ld, row_mul, row_off);
                else place_rows_kernel<__nv_bfloat16><<<grid, 256, 0, m->stream>>>(m->staging, kind, (__nv_bfloat16*)dst, in, out, ld, row_mul, row_off);
                e = cudaGetLastError();
            }
        } else {
            const float scale = std / 65536.0f;
            if (f32) synth_rows_kernel<float><<<grid, 256, 0, m->stream>>>((float*)dst, in, out, ld, row_mul, row_off, key(name), scale);
            else synth_rows_kernel<__nv_bfloat16><<<grid, 256, 0, m->stream>>>((__nv_bfloat16*)dst, in, out, ld, row_mul, row_off, key(name), scale);
            e = cudaGetLastError();
        }
        if (e != cudaSuccess) rc = fail(m, CD_ERR_CUDA, "tensor " + name + ": " + cudaGetErrorString(e));
    }
    // a vector's values; `fill`: its synthetic one
    std::vector<float> values(const std::string& name, std::vector<size_t> shape, float fill) {
        size_t n = 1;
        for (size_t d : shape) n *= d;
        std::vector<float> v(n, fill);
        if (rc || !file) return v;
        const TensorView* t = need(name, shape);
        if (!t) return v;
        for (size_t i = 0; i < n; ++i) {
            if (t->dtype == "F32") memcpy(&v[i], t->data + i * 4, 4);
            else {
                uint16_t u;
                memcpy(&u, t->data + i * 2, 2);
                if (t->dtype == "BF16") { const uint32_t w = (uint32_t)u << 16; memcpy(&v[i], &w, 4); }
                else { __half_raw r; r.x = u; v[i] = __half2float(__half(r)); }
            }
        }
        return v;
    }
    void upload(const std::string& name, void* dst, const void* src, size_t bytes) {
        if (rc) return;
        const cudaError_t e = cudaMemcpy(dst, src, bytes, cudaMemcpyHostToDevice);
        if (e != cudaSuccess) rc = fail(m, CD_ERR_CUDA, "tensor " + name + ": " + cudaGetErrorString(e));
    }
    // a vector to fp32, `add` added to every element (norm weights stored around zero)
    void vector(const std::string& name, float* dst, int n, float add, float fill) {
        std::vector<float> v = values(name, {(size_t)n}, fill);
        for (float& f : v) f += add;
        upload(name, dst, v.data(), (size_t)n * 4);
    }
};

int check_limits(const HybridCfg& h, int dtype) {
    const int kmax = 8 * 256 * (dtype == CD_DTYPE_F32 ? 4 : 8);
    auto unsup = [&](const std::string& msg) { return fail(nullptr, CD_ERR_UNSUPPORTED, h.architecture + ": " + msg); };
    if (h.width > kmax) return unsup("width is limited to " + std::to_string(kmax));
    if (h.side_dim > kmax) return unsup("token side wider than the GEMV tiling");
    for (const auto& L : h.layers) {
        if (L.has_attn() && (L.attn.dim > 256 || L.attn.vdim > 256)) return unsup("attention head widths are limited to 256");
        if (L.has_attn() && pad_to(L.attn.heads * L.attn.vdim, 8) > kmax) return unsup("a mixer's output is wider than the GEMV tiling");
        if (L.has_mem() && pad_to(L.mem.heads * L.mem.vdim, 8) > kmax) return unsup("a mixer's output is wider than the GEMV tiling");
        if (L.mixer == HybridLayerCfg::LATENT) {
            if (pad_to(L.latent.heads * L.latent.vdim, 8) > kmax) return unsup("a mixer's output is wider than the GEMV tiling");
            if (L.latent.rank + L.latent.rot_dim > 1536) return unsup("a latent cache row is limited to 1536 elements");
        }
        if (L.mlp.kind == FfnCfg::DENSE && pad_to(L.mlp.ff, 16) > kmax) return unsup("feed-forward wider than the GEMV tiling");
        if (L.mlp.kind == FfnCfg::MOE && (L.mlp.top > SRC_MAX_LIST || L.mlp.experts > 2048)) return unsup("at most 32 experts per token out of at most 2048");
    }
    return CD_OK;
}

// elements a layer caches per position
size_t cached_elems(const HybridLayerCfg& L) {
    if (L.has_attn()) return (size_t)L.attn.kv_heads * (L.attn.maps * pad_to(L.attn.dim, 16) + pad_to(L.attn.vdim, 16));
    if (L.mixer == HybridLayerCfg::LATENT) return pad_to(L.latent.rank, 16) + pad_to(L.latent.rot_dim, 16);
    return 0;
}

cd_config base_config(const HybridCfg& h, int seq) {
    cd_config c;
    memset(&c, 0, sizeof c);
    const HybridLayerCfg& first = h.layers[0];
    c.dim = h.width;
    c.hidden = 1;
    for (const auto& L : h.layers) c.hidden = std::max(c.hidden, L.mlp.kind == FfnCfg::MOE ? L.mlp.ff * L.mlp.top : L.mlp.ff);
    if (first.has_attn()) { c.heads = first.attn.heads; c.kv_heads = first.attn.kv_heads; c.hd = first.attn.dim; }
    else if (first.has_mem()) { c.heads = c.kv_heads = first.mem.heads; c.hd = first.mem.dim; }
    else { c.heads = c.kv_heads = first.latent.heads; c.hd = first.latent.dim + first.latent.rot_dim; }
    c.seq = seq; c.nlayers = (int)h.layers.size(); c.vocab = h.vocab;
    c.q_dim = c.heads * c.hd; c.kv_dim = c.kv_heads * c.hd; c.gqa_ratio = c.heads / c.kv_heads;
    return c;
}

int build(const std::string& json, const SafeTensors* file, size_t max_tokens, const cd_options* opts_in, uint64_t seed, float std, cd_model** out) {
    HybridCfg h;
    std::string err;
    if (!parse_hybrid_config(json, &h, &err)) return fail(nullptr, CD_ERR_INVALID, err);
    cd_options o;
    memset(&o, 0, sizeof o);
    o.device = -1;
    o.weight_dtype = -1;
    if (opts_in) o = *opts_in;
    if (o.weight_dtype < 0) o.weight_dtype = CD_DTYPE_BF16;
    if (o.weight_dtype != CD_DTYPE_F32 && o.weight_dtype != CD_DTYPE_BF16) return fail(nullptr, CD_ERR_UNSUPPORTED, h.architecture + ": weights are f32 or bf16");
    if (o.tp_world > 1) return fail(nullptr, CD_ERR_UNSUPPORTED, h.architecture + ": one GPU only");
    int rc = check_limits(h, o.weight_dtype);
    if (rc) return rc;
    if (max_tokens == 0) max_tokens = 4096;
    if (max_tokens > (1u << 24)) return fail(nullptr, CD_ERR_INVALID, "max_tokens is limited to 2^24");
    const cd_config cfg = base_config(h, (int)max_tokens);
    const std::vector<LayerRun> runs = h.runs();
    AllocSpec spec;
    spec.family = &HYBRID_FAMILY;
    spec.local = cfg;
    spec.local.dim = pad_to(h.width, 8);
    spec.local.nlayers = (int)runs.size();  // every pass through a layer has cache rows of its own
    for (const LayerRun& r : runs) spec.kv_row_elems.push_back(cached_elems(h.layers[r.layer]));
    cd_model* m = nullptr;
    if ((rc = model_alloc(&cfg, o, h.tied ? 0 : 1, spec, &m))) return rc;
    auto bail = [&](int code) { set_global_error(m->err); cd_model_destroy(m); return code; };
#define CKB(call) do { cudaError_t e_ = (call); if (e_ != cudaSuccess) { fail(m, CD_ERR_CUDA, std::string(#call) + ": " + cudaGetErrorString(e_)); return bail(CD_ERR_CUDA); } } while (0)
    cd_hybrid_state* S = new cd_hybrid_state();
    m->hybrid = S;
    S->cfg = h;
    S->runs = runs;
    m->rms_eps = h.eps;
    m->needs_token = h.side_dim > 0;
    const int width = h.width, D = pad_to(width, 8), nl = (int)h.layers.size();  // rows and vectors are padded with zeros
    const size_t es = esize(o.weight_dtype);
    const int epc = (int)(16 / es);
    S->layers.resize(nl);

    // ---- shapes, then one arena for all layers
    size_t off = 0;
    std::vector<std::pair<void**, size_t>> places;
    auto carve = [&](void** p, size_t bytes) { places.push_back({p, off}); off = align_up(off + bytes, 256); };
    auto mat = [&](void** p, size_t rows, size_t ld) { carve(p, rows * ld * es); };
    auto vec = [&](float** p, size_t n) { carve((void**)p, n * 4); };
    auto norm = [&](VecNorm& v, int kind) {  // weight, and a bias where the kind has one
        v.kind = kind;
        carve((void**)&v.w, (size_t)D * 4);
        if (kind == VecNorm::LAYER) carve((void**)&v.b, (size_t)D * 4);
    };
    const int norm_kind = h.layer_norm ? VecNorm::LAYER : VecNorm::RMS;
    size_t max_proj = 0, max_attn = 1, max_mem = 1, max_gate = 1, max_part = 1, max_ml = 1, max_heads = 1, max_ssq = 1, max_experts = 1, max_qabs = 1, max_qsplit = 1, max_uk = 0;
    for (int l = 0; l < nl; ++l) {
        cd_hybrid_layer& L = S->layers[l];
        L.cfg = h.layers[l];
        const AttnCfg& a = L.cfg.attn;
        const MemCfg& r = L.cfg.mem;
        const LatentCfg& t = L.cfg.latent;
        const FfnCfg& f = L.cfg.mlp;
        ProjLayout& pl = L.proj;
        int at = 0;
        auto take = [&](int n) { const int v = at; at += n; return v; };
        auto rotation = [&](const RotCfg& rot) {
            if (rot.dims > 0) carve((void**)&L.freq, rot.dims / 2 * sizeof(double));
        };
        if (L.cfg.has_attn()) {
            pl.lq = take(a.heads * a.maps * a.dim); pl.lk = take(a.kv_heads * a.maps * a.dim); pl.lv = take(a.kv_heads * a.vdim);
            pl.lg = take(a.gate == AttnCfg::GATE_HEAD ? a.heads : a.gate == AttnCfg::GATE_ELEMENT ? a.heads * a.vdim : 0);
            L.kl = pad_to(a.heads * a.vdim, 8);
            L.ad = AttnDims{a.heads, a.kv_heads, a.dim, a.vdim, pad_to(a.dim, 16), pad_to(a.vdim, 16), a.maps, a.window, m->page_tokens, a.scale, h.eps, a.temp_coef, a.temp_every,
                            a.gate, 0.0f, 1.0f - a.diff, Rotation{nullptr, nullptr, a.rot.dims}};
            if (a.qk_norm) { vec(&L.q_norm, a.heads * a.maps * a.dim); vec(&L.k_norm, a.kv_heads * a.maps * a.dim); }
            if (a.sink) vec(&L.sink, a.heads);
            if (a.distance_bias) vec(&L.slopes, a.heads);
            rotation(a.rot);
            max_attn = std::max<size_t>(max_attn, L.kl);
        }
        if (L.cfg.has_mem()) {
            const bool matrix = r.kind == MemCfg::MATRIX;
            pl.rq = take(r.heads * r.dim); pl.rk = take(r.heads * r.dim); pl.rv = take(r.heads * r.vdim); pl.rg = take(r.heads * r.vdim);
            if (matrix) { pl.ri = take(r.heads); pl.rf = take(r.heads); vec(&L.ib, r.heads); vec(&L.fb, r.heads); }
            else { vec(&L.decay, r.heads); vec(&L.log_decay, r.heads); }
            L.kr = pad_to(r.heads * r.vdim, 8);
            L.md = MemDims{r.heads, r.dim, r.vdim, pad_to(r.vdim, 4), (r.vdim + MEM_SLICE - 1) / MEM_SLICE, r.gate_cap, h.eps, nullptr, nullptr};
            vec(&L.mem_norm, r.heads * r.vdim);
            max_mem = std::max<size_t>(max_mem, L.kr);
            max_ssq = std::max<size_t>(max_ssq, (size_t)r.heads * L.md.nslice);
            if (L.cfg.mixer == HybridLayerCfg::MEMORY) { L.kl = L.kr; L.kr = 0; }
        }
        if (L.cfg.mixer == HybridLayerCfg::LATENT) {
            pl.lq = take(t.heads * (t.dim + t.rot_dim) + t.rank + t.rot_dim);
            L.kl = pad_to(t.heads * t.vdim, 8);
            L.ld = MlaDims{t.heads, pad_to(t.rank, 16), pad_to(t.rot_dim, 16), pad_to(t.dim, epc), t.vdim, m->page_tokens, t.rank, t.rot_dim, t.dim, t.rot.dims, t.window, h.eps};
            mat(&L.wuk_t, (size_t)t.heads * L.ld.latent, L.ld.nope);
            const size_t key_rows = o.weight_dtype == CD_DTYPE_F32 ? 0 : (size_t)t.heads * t.dim;  // the prompt pass expands keys, too
            mat(&L.wukv, key_rows + (size_t)t.heads * t.vdim, L.ld.latent);
            max_uk = std::max<size_t>(max_uk, (size_t)t.heads * t.dim * t.rank);
            vec(&L.latent_norm, t.rank);
            rotation(t.rot);
            max_attn = std::max<size_t>(max_attn, L.kl);
            max_qabs = std::max<size_t>(max_qabs, (size_t)t.heads * L.ld.row());
            max_qsplit = std::max<size_t>(max_qsplit, (size_t)L.ld.head_blocks() * 32 * L.ld.row());
        }
        pl.rows = at;
        L.ffp = f.kind == FfnCfg::NONE ? 0 : pad_to(f.ff, 16);
        // slices of whole tiles of the visible positions, as many as one wave of CTAs has room for beside a memory's
        const int window = L.cfg.has_attn() ? a.window : t.window;
        const size_t seen = window > 0 ? std::min<size_t>(window, max_tokens) : max_tokens;
        if (L.cfg.has_attn()) {
            const int tiles = (int)((seen + MIX_TILE - 1) / MIX_TILE), room = std::max(1, (4 * m->sm_count - L.md.H * L.md.nslice) / a.heads);
            const int per_slice = std::max((tiles + 31) / 32, (tiles + room - 1) / room);
            L.nsplit = std::max(1, (tiles + per_slice - 1) / per_slice);
            max_part = std::max<size_t>(max_part, (size_t)a.heads * a.maps * L.nsplit * L.ad.vp);
            max_ml = std::max<size_t>(max_ml, (size_t)a.heads * a.maps * L.nsplit * 2);
            max_heads = std::max<size_t>(max_heads, a.heads);
        } else if (L.cfg.mixer == HybridLayerCfg::LATENT) {
            L.nsplit = (int)std::max<size_t>(1, std::min<size_t>(64, (seen + MLA_MMA_TILE - 1) / MLA_MMA_TILE));
            max_part = std::max<size_t>(max_part, (size_t)t.heads * L.nsplit * L.ld.latent);
            max_ml = std::max<size_t>(max_ml, (size_t)t.heads * L.nsplit * 2);
        }
        mat(&L.wmix, pl.rows, D); mat(&L.wo_l, D, L.kl);
        if (L.cfg.mixer == HybridLayerCfg::PARALLEL) { mat(&L.wo_r, D, L.kr); vec(&L.out_l, D); vec(&L.out_r, D); }
        if (h.pre_norms) norm(L.pre1, norm_kind);
        norm(L.post1, norm_kind);
        const size_t nm = f.kind == FfnCfg::MOE ? f.experts : 1;
        if (f.kind != FfnCfg::NONE) {
            mat(&L.w13, nm * 2 * L.ffp, D); mat(&L.w2, nm * D, L.ffp);
            if (h.pre_norms) norm(L.pre2, norm_kind);
            norm(L.post2, norm_kind);
        }
        if (f.kind == FfnCfg::MOE) {
            mat(&L.wr, f.experts, D);
            const size_t units = (size_t)f.top * L.ffp;
            L.stream_ffn = (units / epc + 255) / 256 <= 8 && units * es * 2 <= (size_t)180 * 1024;  // a thread's share of the widest row fits its registers, two rows the ring
            max_experts = std::max<size_t>(max_experts, f.experts);
        }
        if (h.side_dim) {
            mat(&L.side_gate, h.side_dim, D); mat(&L.side_proj, D, S->side_pad());
            norm(L.side_norm, VecNorm::RMS);
        }
        max_proj = std::max<size_t>(max_proj, pl.rows);
        max_gate = std::max<size_t>(max_gate, (size_t)L.ffp * (f.kind == FfnCfg::MOE ? f.top : 1));
    }
    if (h.side_dim) mat(&S->side_embed, h.vocab, S->side_ld());
    if (h.loop_times) vec(&S->loop_step, (size_t)h.loop_times * D);
    S->final_norm = VecNorm{norm_kind, m->gamma_final, nullptr};
    if (h.layer_norm) carve((void**)&S->final_norm.b, (size_t)D * 4);
    CKB(cudaMalloc(&m->layer_arena, off));
    CKB(cudaMemsetAsync(m->layer_arena, 0, off, m->stream));
    for (auto& pr : places) *pr.first = (char*)m->layer_arena + pr.second;
    m->weight_bytes += off;
    for (auto& L : S->layers) {
        L.md.decay = L.decay;
        L.md.log_decay = L.log_decay;
        L.ad.rot.freq = L.freq;
        if (L.wukv) L.wuv = (char*)L.wukv + (o.weight_dtype == CD_DTYPE_F32 ? 0 : (size_t)L.ld.heads * L.ld.nope_n * L.ld.latent * es);
    }
    size_t state = 0;
    for (const LayerRun& r : runs) {
        S->state_off.push_back(state);
        if (S->layers[r.layer].cfg.has_mem()) state += S->layers[r.layer].md.floats();
    }
    S->slot_floats = state;
    CKB(cudaMalloc(&S->state, std::max<size_t>(cd_hybrid_state::SLOTS * state * 4, 256)));
    CKB(cudaMemsetAsync(S->state, 0, cd_hybrid_state::SLOTS * state * 4, m->stream));
    // ---- scratch of a step
    off = 0;
    places.clear();
    vec(&S->proj, max_proj); vec(&S->attn, max_attn); vec(&S->mem, max_mem); vec(&S->ssq, max_ssq); vec(&S->y, 2 * (size_t)D); vec(&S->y2, D);
    vec(&S->gate, max_gate); vec(&S->side, S->side_pad()); vec(&S->part_acc, max_part); vec(&S->part_ml, max_ml); vec(&S->router_logits, max_experts);
    vec(&S->sel_w, SRC_MAX_LIST); vec(&S->loc_w, SRC_MAX_LIST); vec(&S->zero, D); vec(&S->qabs, max_qabs); carve(&S->qsplit, max_qsplit * 2);
    carve((void**)&S->counters, max_heads * 4); carve((void**)&S->router_counter, 4);
    carve((void**)&S->sel_ids, (size_t)nl * SRC_MAX_LIST * 4); carve((void**)&S->loc_ids, SRC_MAX_LIST * 4); carve((void**)&S->n_loc, 4);
    CKB(cudaMalloc(&S->ws, off));
    CKB(cudaMemsetAsync(S->ws, 0, off, m->stream));
    for (auto& pr : places) *pr.first = (char*)S->ws + pr.second;
    void* uk_raw = nullptr;  // a layer's key matrix as stored, ahead of its transposition
    if (max_uk) {
        CKB(cudaMalloc(&uk_raw, max_uk * es));
        m->staging2 = uk_raw;  // freed with the other upload buffers
    }
    CKB(cudaStreamSynchronize(m->stream));

    // ---- tensors
    TensorSource T;
    T.file = file; T.seed = seed; T.std = std; T.m = m;
    auto load_norm = [&](const std::string& name, const VecNorm& v, bool around_zero) {
        if (!v.w) return;
        T.vector(name, const_cast<float*>(v.w), width, around_zero ? 1.0f : 0.0f, around_zero ? 0.0f : 1.0f);
        if (v.b) T.vector(name + ".b", const_cast<float*>(v.b), width, 0.0f, 0.0f);
    };
    T.matrix("embed", m->embed, h.vocab, width, D);
    if (!h.tied) T.matrix("head", m->lm_head, h.vocab, width, D);
    load_norm("final.norm", S->final_norm, !h.layer_norm);
    if (h.side_dim) T.matrix("side.embed", S->side_embed, h.vocab, S->side_ld(), S->side_ld());
    if (h.loop_times) {
        const std::vector<float> v = T.values("loop.step", {(size_t)h.loop_times, (size_t)width}, 0.0f);
        for (int t = 0; t < h.loop_times; ++t) T.upload("loop.step", S->loop_step + (size_t)t * D, v.data() + (size_t)t * width, (size_t)width * 4);
    }
    for (int l = 0; l < nl && !T.rc; ++l) {
        cd_hybrid_layer& L = S->layers[l];
        const AttnCfg& a = L.cfg.attn;
        const MemCfg& r = L.cfg.mem;
        const LatentCfg& t = L.cfg.latent;
        const FfnCfg& f = L.cfg.mlp;
        const bool pair = L.cfg.mixer == HybridLayerCfg::PARALLEL;
        const std::string p = "l" + std::to_string(l) + ".", pl = p + (pair ? "mix.left." : "mix."), pr = p + (pair ? "mix.right." : "mix."), pm = p + "mlp.";
        auto rows = [&](const std::string& name, int first, int n) { T.matrix(name, (char*)L.wmix + (size_t)first * D * es, n, width, D); };
        auto rotation = [&](const RotCfg& rot) {
            const std::vector<double> v = rot_frequencies(rot);
            if (!v.empty()) T.upload(p + "rotation", L.freq, v.data(), v.size() * sizeof(double));
        };
        if (L.cfg.has_attn()) {
            rows(pl + "q", L.proj.lq, a.heads * a.maps * a.dim); rows(pl + "k", L.proj.lk, a.kv_heads * a.maps * a.dim); rows(pl + "v", L.proj.lv, a.kv_heads * a.vdim);
            if (a.gate != AttnCfg::GATE_NONE) rows(pl + "g", L.proj.lg, a.gate == AttnCfg::GATE_HEAD ? a.heads : a.heads * a.vdim);
            T.matrix(pl + "o", L.wo_l, width, a.heads * a.vdim, L.kl);
            if (a.qk_norm) { T.vector(pl + "q.norm", L.q_norm, a.heads * a.dim, 0.f, 1.f); T.vector(pl + "k.norm", L.k_norm, a.kv_heads * a.dim, 0.f, 1.f); }
            if (a.sink) T.vector(pl + "sink", L.sink, a.heads, 0.f, 0.f);
            if (a.distance_bias) {  // slopes 2^(-8 (h + 1) / H)
                std::vector<float> sl(a.heads);
                for (int i = 0; i < a.heads; ++i) sl[i] = (float)std::pow(2.0, -8.0 * (i + 1) / a.heads);
                T.upload(pl + "slopes", L.slopes, sl.data(), sl.size() * 4);
            }
            rotation(a.rot);
            if (a.maps == 2) {  // the second map's weight: one number for the layer
                auto dot = [&](const char* u, const char* v) {
                    const std::vector<float> x = T.values(pl + u, {(size_t)a.dim}, 0.f), y = T.values(pl + v, {(size_t)a.dim}, 0.f);
                    double s = 0.0;
                    for (int i = 0; i < a.dim; ++i) s += (double)x[i] * y[i];
                    return s;
                };
                L.ad.lambda = (float)(std::exp(dot("lq1", "lk1")) - std::exp(dot("lq2", "lk2")) + a.diff);
            }
        }
        if (L.cfg.has_mem()) {
            rows(pr + "q", L.proj.rq, r.heads * r.dim); rows(pr + "k", L.proj.rk, r.heads * r.dim); rows(pr + "v", L.proj.rv, r.heads * r.vdim);
            rows(pr + "g", L.proj.rg, r.heads * r.vdim);
            if (r.kind == MemCfg::MATRIX) {
                rows(pr + "i", L.proj.ri, r.heads); rows(pr + "f", L.proj.rf, r.heads);
                T.vector(pr + "i.b", L.ib, r.heads, 0.f, 0.f); T.vector(pr + "f.b", L.fb, r.heads, 0.f, 3.f);
            } else {
                std::vector<float> d(r.heads), ld(r.heads);
                for (int i = 0; i < r.heads; ++i) {
                    d[i] = (float)r.decay[i];
                    ld[i] = (float)std::max(std::log(std::max(r.decay[i], 1e-300)), -200.0);  // exp(-200) is zero in fp32
                }
                T.upload(pr + "decay", L.decay, d.data(), d.size() * 4);
                T.upload(pr + "decay", L.log_decay, ld.data(), ld.size() * 4);
            }
            T.vector(pr + "norm", L.mem_norm, r.heads * r.vdim, 0.f, 1.f);
            T.matrix(pr + "o", pair ? L.wo_r : L.wo_l, width, r.heads * r.vdim, pair ? L.kr : L.kl);
        }
        if (pair) { T.vector(pl + "out", L.out_l, width, 0.f, 1.f); T.vector(pr + "out", L.out_r, width, 0.f, 1.f); }
        if (L.cfg.mixer == HybridLayerCfg::LATENT) {
            const int nq = t.heads * (t.dim + t.rot_dim), C = L.ld.latent;
            rows(pl + "q", 0, nq); rows(pl + "dkv", nq, t.rank + t.rot_dim);
            T.vector(pl + "dkv.norm", L.latent_norm, t.rank, 0.f, 1.f);
            rotation(t.rot);
            T.matrix(pl + "uk", uk_raw, t.heads * t.dim, t.rank, t.rank);
            if (!T.rc) {
                const int grid = m->sm_count * 4;
                if (o.weight_dtype == CD_DTYPE_F32) transpose_heads_kernel<float><<<grid, 256, 0, m->stream>>>((const float*)uk_raw, (float*)L.wuk_t, t.heads, t.dim, t.rank, t.rank, C, L.ld.nope);
                else transpose_heads_kernel<__nv_bfloat16><<<grid, 256, 0, m->stream>>>((const __nv_bfloat16*)uk_raw, (__nv_bfloat16*)L.wuk_t, t.heads, t.dim, t.rank, t.rank, C, L.ld.nope);
                const cudaError_t e = cudaGetLastError();
                if (e != cudaSuccess) T.rc = fail(m, CD_ERR_CUDA, "tensor " + pl + "uk: " + cudaGetErrorString(e));
            }
            if (o.weight_dtype != CD_DTYPE_F32) T.matrix(pl + "uk", L.wukv, t.heads * t.dim, t.rank, C);
            T.matrix(pl + "uv", L.wuv, t.heads * t.vdim, t.rank, C);
            T.matrix(pl + "o", L.wo_l, width, t.heads * t.vdim, L.kl);
        }
        // with norms ahead of the sublayers those are "norm1", "norm2" and the ones behind have a b; without, the plain names
        load_norm(p + "norm1", L.pre1, !h.layer_norm);
        load_norm(p + (h.pre_norms ? "norm1b" : "norm1"), L.post1, !h.layer_norm);
        if (h.side_dim) {
            T.matrix(p + "side.gate", L.side_gate, h.side_dim, width, D);
            T.matrix(p + "side.proj", L.side_proj, width, h.side_dim, S->side_pad());
            load_norm(p + "side.norm", L.side_norm, false);
        }
        if (f.kind == FfnCfg::NONE) continue;
        load_norm(p + "norm2", L.pre2, !h.layer_norm);
        load_norm(p + (h.pre_norms ? "norm2b" : "norm2"), L.post2, !h.layer_norm);
        auto ffn = [&](const std::string& q, size_t i) {
            char* w13 = (char*)L.w13 + i * 2 * L.ffp * D * es;
            T.matrix(q + "gate", w13, f.ff, width, D, 2, 0);
            T.matrix(q + "up", w13, f.ff, width, D, 2, 1);
            T.matrix(q + "down", (char*)L.w2 + i * D * L.ffp * es, width, f.ff, L.ffp);
        };
        if (f.kind == FfnCfg::DENSE) {
            ffn(pm, 0);
        } else {
            T.matrix(pm + "router", L.wr, f.experts, width, D);
            for (int i = 0; i < f.experts; ++i) ffn(pm + "e" + std::to_string(i) + ".", (size_t)i);
        }
    }
    if (T.rc) return bail(T.rc);
    if ((rc = model_finish(m))) return bail(rc);
    *out = m;
    return CD_OK;
#undef CKB
}

bool read_text(const std::string& path, std::string* out) {
    std::ifstream f(path, std::ios::binary);
    if (!f) return false;
    out->assign(std::istreambuf_iterator<char>(f), std::istreambuf_iterator<char>());
    return true;
}

}  // namespace

extern "C" {

int cd_model_create_from_dir(const char* dir, size_t max_tokens, const cd_options* opts, cd_model** out) {
    if (!dir || !out) return fail(nullptr, CD_ERR_INVALID, "null argument");
    *out = nullptr;
    std::string json, err;
    if (!read_text(std::string(dir) + "/config.json", &json)) return fail(nullptr, CD_ERR_IO, std::string("cannot read ") + dir + "/config.json");
    SafeTensors file;
    if (!file.open(std::string(dir) + "/model.safetensors", &err)) return fail(nullptr, CD_ERR_IO, err);
    return build(json, &file, max_tokens, opts, 0, 0.f, out);
}

int cd_model_create_from_config(const char* config_json, size_t max_tokens, const cd_options* opts, uint64_t seed, float std, cd_model** out) {
    if (!config_json || !out) return fail(nullptr, CD_ERR_INVALID, "null argument");
    *out = nullptr;
    return build(config_json, nullptr, max_tokens, opts, seed, std, out);
}

int cd_config_info(const char* config_json, cd_config* cfg_out) {
    if (!config_json || !cfg_out) return fail(nullptr, CD_ERR_INVALID, "null argument");
    HybridCfg h;
    std::string err;
    if (!parse_hybrid_config(config_json, &h, &err)) return fail(nullptr, CD_ERR_INVALID, err);
    *cfg_out = base_config(h, 0);
    return CD_OK;
}

}  // extern "C"
