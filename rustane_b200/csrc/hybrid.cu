// The configured decoder family (hybrid.h): construction from a model folder (config.json + model.safetensors) or from a
// configuration with synthetic weights, the per-token step, and the recurrent state's snapshots.
//
// A step, per layer (each line a kernel of the token's chain, programmatic dependent launch between them):
//   gemv_tma_kernel     every projection of the mixer's input; its prologue forms the residual stream behind the
//                       previous sublayer (InNormedResidual / InParallelMix)
//   mixer_step_kernel   both mixers, cache append, state update
//   gemv_tma_kernel     both output projections in one launch (SrcPair, InMixerOutputs)
//   gemv_tma_kernel     gate | up with the mixers' norms and residual in its prologue; for a mixture of experts
//                       moe_router_kernel does that and the chosen experts' rows are gathered (SrcExpertRows)
//   gemv_tma_kernel     down (SrcExpertCols)
#include <algorithm>
#include <cmath>
#include <cstring>
#include <fstream>
#include <iterator>
#include <memory>

#include "step.cuh"
#include "moe.cuh"
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
    const int D = c.dim;
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
    const cd_hybrid_layer* behind = nullptr;  // the layer whose last sublayer's output is still to be added
    float *yl = S.y, *yr = S.y + D;
    auto ffn_in = [&](const cd_hybrid_layer& L) { return InNormedResidual{x[cur], S.y2, L.gain2, x[cur ^ 1], mult, eps, D}; };
    auto mix_in = [&](const cd_hybrid_layer& L) { return InParallelMix{x[cur], yl, yr, L.out_l, L.out_r, L.gain1, x[cur ^ 1], mult, eps, D}; };
    // the next GEMV's first rows, pulled into L2 behind a GEMV's own last loads
    auto hint = [&](const void* w, int K, int N, int unit) {
        m->next_stream = NextStream{m->prefetch_kb > 0 ? w : nullptr, Wfmt<WT>::row_stride(K), N / unit, unit, (uint32_t)m->prefetch_kb * 1024u};
    };
    for (int l = 0; l < c.nlayers; ++l) {
        const cd_hybrid_layer& L = S.layers[l];
        const cd_hybrid_layer* next = l + 1 < c.nlayers ? &S.layers[l + 1] : nullptr;
        auto hint_next = [&]() {
            if (next) hint(next->wmix, D, next->proj.rows, 1);
            else if (p.head != HEAD_NONE) hint(m->lm_head, D, m->v_loc, 1);
        };
        m->cur_cls = CLS_QKV;
        const EpiStore to_proj{S.proj};
        if (!behind) {
            TRY((launch_gemv<WT, 1, false>(m, L.wmix, x[cur], nullptr, nullptr, L.proj.rows, D, to_proj)));
        } else if (behind->cfg.mlp.kind != FfnCfg::NONE) {
            TRY((launch_gemv<WT, 1, false>(m, L.wmix, x[cur], nullptr, nullptr, L.proj.rows, D, to_proj, SrcPlain{}, ffn_in(*behind))));
            cur ^= 1;
        } else {
            TRY((launch_gemv<WT, 1, false>(m, L.wmix, x[cur], nullptr, nullptr, L.proj.rows, D, to_proj, SrcPlain{}, mix_in(*behind))));
            cur ^= 1;
        }
        behind = &L;
        m->cur_cls = CLS_ATTN;
        {
            MixerStep q;
            q.a = L.ad; q.d = L.md; q.pl = L.proj; q.proj = S.proj;
            q.q_norm = L.q_norm; q.k_norm = L.k_norm; q.sink = L.sink; q.slopes = L.slopes; q.ib = L.ib; q.fb = L.fb;
            q.page_table = m->page_table; q.st = m->st;
            q.part_acc = S.part_acc; q.part_ml = S.part_ml; q.counters = S.counters;
            q.attn = S.attn; q.mem = S.mem; q.ssq = S.ssq; q.state = S.state + L.state_off; q.nsplit = L.nsplit;
            const size_t smem = std::max(mixer_attn_smem_floats(L.ad.kp, L.ad.vp), mixer_mem_smem_floats(L.md.dim)) * sizeof(float);
            static size_t smem_set = 48 * 1024;  // per instantiation
            if (smem > smem_set) {
                TRY(cudaFuncSetAttribute(mixer_step_kernel<KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
                smem_set = smem;
            }
            TRY(launch_chain(m, mixer_step_kernel<KT>, dim3(L.md.H * L.md.nslice + L.ad.H * L.nsplit), dim3(MIX_THREADS), smem, q, (KT*)m->layers[l].kv));
        }
        m->cur_cls = CLS_WO;
        {
            if (L.cfg.mlp.kind == FfnCfg::DENSE) hint(L.w13, D, 2 * L.ffp, 2);
            else if (L.cfg.mlp.kind == FfnCfg::NONE) hint_next();
            const InMixerOutputs in{S.attn, S.mem, S.ssq, L.mem_norm, S.proj + L.proj.rg, L.md.H * L.md.vdim, L.md.vdim, L.md.nslice, eps};
            TRY((launch_gemv<WT, 1, false>(m, L.wo_l, S.attn, nullptr, nullptr, D, L.kl, EpiStore{S.y}, SrcPair{L.wo_r, D, L.kr, 0}, in)));
        }
        const FfnCfg& f = L.cfg.mlp;
        if (f.kind == FfnCfg::DENSE) {
            m->cur_cls = CLS_W13;
            hint(L.w2, L.ffp, D, 1);
            TRY((launch_gemv<WT, 2, false>(m, L.w13, x[cur], nullptr, nullptr, 2 * L.ffp, D, EpiGate{S.gate, CD_ACT_SWIGLU}, SrcPlain{}, mix_in(L))));
            cur ^= 1;
            m->cur_cls = CLS_W2;
            hint_next();
            TRY((launch_gemv<WT, 1, false>(m, L.w2, S.gate, nullptr, nullptr, D, L.ffp, EpiStore{S.y2})));
        } else if (f.kind == FfnCfg::MOE) {
            m->cur_cls = CLS_W13;
            int* sel = S.sel_ids + (size_t)l * SRC_MAX_LIST;
            TRY(launch_chain(m, moe_router_kernel<WT, RouterMixIn>, dim3((f.experts + 3) / 4), dim3(128), (size_t)std::max(D, f.experts + f.groups) * sizeof(float),
                             RouterMixIn{x[cur], yl, yr, L.out_l, L.out_r, L.gain1, x[cur ^ 1], mult, eps}, (const WT*)L.wr, S.router_logits, S.router_counter, sel,
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
    }
    m->cur_cls = CLS_MISC;
    if (behind->cfg.mlp.kind != FfnCfg::NONE) {
        InNormedResidual in = ffn_in(*behind);
        in.x_out = m->x_a;
        TRY(launch_chain(m, vector_input_kernel<InNormedResidual>, dim3(1), dim3(GEMV_CONSUMERS), 0, in, D));
    } else {
        InParallelMix in = mix_in(*behind);
        in.x_out = m->x_a;
        TRY(launch_chain(m, vector_input_kernel<InParallelMix>, dim3(1), dim3(GEMV_CONSUMERS), 0, in, D));
    }
    return enqueue_head_t<WT, WT>(m, p, false, 0u, 0);
#undef TRY
}

cudaError_t hybrid_step(cd_model* m, const cd_step& p) {
    if (m->opt.weight_dtype == CD_DTYPE_F32) return hybrid_step_t<float, float>(m, p);
    return m->kv_dtype == CD_DTYPE_F16 ? hybrid_step_t<__nv_bfloat16, __half>(m, p) : hybrid_step_t<__nv_bfloat16, __nv_bfloat16>(m, p);
}

cudaError_t hybrid_head_only(cd_model* m) {
    return m->opt.weight_dtype == CD_DTYPE_F32 ? enqueue_head_only_t<float>(m) : enqueue_head_only_t<__nv_bfloat16>(m);
}

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
    // a vector to fp32, `add` added to every element (norm weights stored around zero); `fill`: its synthetic value
    void vector(const std::string& name, float* dst, int n, float add, float fill) {
        if (rc) return;
        std::vector<float> v(n, fill);
        if (file) {
            const TensorView* t = need(name, {(size_t)n});
            if (!t) return;
            for (int i = 0; i < n; ++i) {
                if (t->dtype == "F32") memcpy(&v[i], t->data + (size_t)i * 4, 4);
                else {
                    uint16_t u;
                    memcpy(&u, t->data + (size_t)i * 2, 2);
                    if (t->dtype == "BF16") { const uint32_t w = (uint32_t)u << 16; memcpy(&v[i], &w, 4); }
                    else { __half_raw r; r.x = u; v[i] = __half2float(__half(r)); }
                }
            }
        }
        for (float& f : v) f += add;
        const cudaError_t e = cudaMemcpy(dst, v.data(), (size_t)n * 4, cudaMemcpyHostToDevice);
        if (e != cudaSuccess) rc = fail(m, CD_ERR_CUDA, "tensor " + name + ": " + cudaGetErrorString(e));
    }
};

int check_limits(const HybridCfg& h, int dtype) {
    const int kmax = 8 * 256 * (dtype == CD_DTYPE_F32 ? 4 : 8);
    auto unsup = [&](const std::string& msg) { return fail(nullptr, CD_ERR_UNSUPPORTED, h.architecture + ": " + msg); };
    if (h.width % 8 || h.width > kmax) return unsup("width must be a multiple of 8 and at most " + std::to_string(kmax));
    for (const auto& L : h.layers) {
        if (L.left.dim > 256 || L.left.vdim > 256) return unsup("attention head widths are limited to 256");
        if (pad_to(L.left.heads * L.left.vdim, 8) > kmax || pad_to(L.right.heads * L.right.vdim, 8) > kmax) return unsup("a mixer's output is wider than the GEMV tiling");
        if (L.mlp.kind == FfnCfg::DENSE && pad_to(L.mlp.ff, 16) > kmax) return unsup("feed-forward wider than the GEMV tiling");
        if (L.mlp.kind == FfnCfg::MOE && (L.mlp.top > SRC_MAX_LIST || L.mlp.experts > 2048)) return unsup("at most 32 experts per token out of at most 2048");
    }
    return CD_OK;
}

cd_config base_config(const HybridCfg& h, int seq) {
    cd_config c;
    memset(&c, 0, sizeof c);
    const AttnCfg& a = h.layers[0].left;
    c.dim = h.width;
    c.hidden = 1;
    for (const auto& L : h.layers) c.hidden = std::max(c.hidden, L.mlp.kind == FfnCfg::MOE ? L.mlp.ff * L.mlp.top : L.mlp.ff);
    c.heads = a.heads; c.kv_heads = a.kv_heads; c.hd = a.dim; c.seq = seq; c.nlayers = (int)h.layers.size(); c.vocab = h.vocab;
    c.q_dim = a.heads * a.dim; c.kv_dim = a.kv_heads * a.dim; c.gqa_ratio = a.heads / a.kv_heads;
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
    AllocSpec spec;
    spec.family = &HYBRID_FAMILY;
    spec.local = cfg;
    for (const auto& L : h.layers) spec.kv_row_elems.push_back((size_t)L.left.kv_heads * (pad_to(L.left.dim, 16) + pad_to(L.left.vdim, 16)));
    cd_model* m = nullptr;
    if ((rc = model_alloc(&cfg, o, 1, spec, &m))) return rc;
    auto bail = [&](int code) { set_global_error(m->err); cd_model_destroy(m); return code; };
#define CKB(call) do { cudaError_t e_ = (call); if (e_ != cudaSuccess) { fail(m, CD_ERR_CUDA, std::string(#call) + ": " + cudaGetErrorString(e_)); return bail(CD_ERR_CUDA); } } while (0)
    cd_hybrid_state* S = new cd_hybrid_state();
    m->hybrid = S;
    S->cfg = h;
    m->rms_eps = h.eps;
    const int D = h.width, nl = (int)h.layers.size();
    const size_t es = esize(o.weight_dtype);
    S->layers.resize(nl);

    // ---- shapes, then one arena for all layers
    size_t off = 0;
    std::vector<std::pair<void**, size_t>> places;
    auto carve = [&](void** p, size_t bytes) { places.push_back({p, off}); off = align_up(off + bytes, 256); };
    auto mat = [&](void** p, size_t rows, size_t ld) { carve(p, rows * ld * es); };
    auto vec = [&](float** p, size_t n) { carve((void**)p, n * 4); };
    size_t state = 0, max_proj = 0, max_kl = 0, max_kr = 0, max_gate = 1, max_part = 0, max_heads = 0, max_ssq = 0, max_experts = 1;
    for (int l = 0; l < nl; ++l) {
        cd_hybrid_layer& L = S->layers[l];
        L.cfg = h.layers[l];
        const AttnCfg& a = L.cfg.left;
        const MemCfg& r = L.cfg.right;
        const FfnCfg& f = L.cfg.mlp;
        ProjLayout& pl = L.proj;
        int at = 0;
        auto take = [&](int n) { const int v = at; at += n; return v; };
        pl.lq = take(a.heads * a.dim); pl.lk = take(a.kv_heads * a.dim); pl.lv = take(a.kv_heads * a.vdim); pl.lg = take(a.heads);
        pl.rq = take(r.heads * r.dim); pl.rk = take(r.heads * r.dim); pl.rv = take(r.heads * r.vdim); pl.rg = take(r.heads * r.vdim);
        pl.ri = take(r.heads); pl.rf = take(r.heads);
        pl.rows = at;
        L.kl = pad_to(a.heads * a.vdim, 8);
        L.kr = pad_to(r.heads * r.vdim, 8);
        L.ffp = f.kind == FfnCfg::NONE ? 0 : pad_to(f.ff, 16);
        L.ad = AttnDims{a.heads, a.kv_heads, a.dim, a.vdim, pad_to(a.dim, 16), pad_to(a.vdim, 16), a.window, m->page_tokens, a.scale, h.eps, a.temp_coef, a.temp_every};
        L.md = MemDims{r.heads, r.dim, r.vdim, pad_to(r.vdim, 4), (r.vdim + MEM_SLICE - 1) / MEM_SLICE, r.gate_cap, h.eps};
        const size_t seen = a.window > 0 ? std::min<size_t>(a.window, max_tokens) : max_tokens;
        // slices of whole tiles, as many as one wave of CTAs has room for beside the memory's
        const int tiles = (int)((seen + MIX_TILE - 1) / MIX_TILE), room = std::max(1, (4 * m->sm_count - L.md.H * L.md.nslice) / a.heads);
        const int per_slice = std::max((tiles + 31) / 32, (tiles + room - 1) / room);
        L.nsplit = std::max(1, (tiles + per_slice - 1) / per_slice);
        L.state_off = state;
        state += L.md.floats();
        mat(&L.wmix, pl.rows, D); mat(&L.wo_l, D, L.kl); mat(&L.wo_r, D, L.kr);
        vec(&L.q_norm, a.heads * a.dim); vec(&L.k_norm, a.kv_heads * a.dim); vec(&L.sink, a.heads); vec(&L.slopes, a.heads);
        vec(&L.mem_norm, r.heads * r.vdim); vec(&L.ib, r.heads); vec(&L.fb, r.heads);
        vec(&L.out_l, D); vec(&L.out_r, D); vec(&L.gain1, D);
        const size_t nm = f.kind == FfnCfg::MOE ? f.experts : 1;
        if (f.kind != FfnCfg::NONE) {
            mat(&L.w13, nm * 2 * L.ffp, D); mat(&L.w2, nm * D, L.ffp);
            vec(&L.gain2, D);
        }
        if (f.kind == FfnCfg::MOE) {
            mat(&L.wr, f.experts, D);
            const size_t epc = 16 / es, units = (size_t)f.top * L.ffp;
            L.stream_ffn = (units / epc + 255) / 256 <= 8 && units * es * 2 <= (size_t)180 * 1024;  // a thread's share of the widest row fits its registers, two rows the ring
            max_experts = std::max<size_t>(max_experts, f.experts);
        }
        max_proj = std::max<size_t>(max_proj, pl.rows); max_kl = std::max<size_t>(max_kl, L.kl); max_kr = std::max<size_t>(max_kr, L.kr);
        max_gate = std::max<size_t>(max_gate, (size_t)L.ffp * (f.kind == FfnCfg::MOE ? f.top : 1));
        max_part = std::max<size_t>(max_part, (size_t)a.heads * L.nsplit * L.ad.vp); max_heads = std::max<size_t>(max_heads, a.heads);
        max_ssq = std::max<size_t>(max_ssq, (size_t)r.heads * L.md.nslice);
    }
    CKB(cudaMalloc(&m->layer_arena, off));
    CKB(cudaMemsetAsync(m->layer_arena, 0, off, m->stream));
    for (auto& pr : places) *pr.first = (char*)m->layer_arena + pr.second;
    m->weight_bytes += off;
    S->slot_floats = state;
    CKB(cudaMalloc(&S->state, cd_hybrid_state::SLOTS * state * 4));
    CKB(cudaMemsetAsync(S->state, 0, cd_hybrid_state::SLOTS * state * 4, m->stream));
    // ---- scratch of a step
    off = 0;
    places.clear();
    vec(&S->proj, max_proj); vec(&S->attn, max_kl); vec(&S->mem, max_kr); vec(&S->ssq, max_ssq); vec(&S->y, 2 * (size_t)D); vec(&S->y2, D);
    vec(&S->gate, max_gate); vec(&S->part_acc, max_part); vec(&S->part_ml, max_heads * 32 * 2); vec(&S->router_logits, max_experts);
    vec(&S->sel_w, SRC_MAX_LIST); vec(&S->loc_w, SRC_MAX_LIST); vec(&S->zero, D);
    carve((void**)&S->counters, max_heads * 4); carve((void**)&S->router_counter, 4);
    carve((void**)&S->sel_ids, (size_t)nl * SRC_MAX_LIST * 4); carve((void**)&S->loc_ids, SRC_MAX_LIST * 4); carve((void**)&S->n_loc, 4);
    CKB(cudaMalloc(&S->ws, off));
    CKB(cudaMemsetAsync(S->ws, 0, off, m->stream));
    for (auto& pr : places) *pr.first = (char*)S->ws + pr.second;
    CKB(cudaStreamSynchronize(m->stream));

    // ---- tensors
    TensorSource T;
    T.file = file; T.seed = seed; T.std = std; T.m = m;
    T.matrix("embed", m->embed, h.vocab, D, D);
    T.matrix("head", m->lm_head, h.vocab, D, D);
    T.vector("final.norm", m->gamma_final, D, 1.0f, 0.0f);
    for (int l = 0; l < nl && !T.rc; ++l) {
        cd_hybrid_layer& L = S->layers[l];
        const AttnCfg& a = L.cfg.left;
        const MemCfg& r = L.cfg.right;
        const FfnCfg& f = L.cfg.mlp;
        const std::string p = "l" + std::to_string(l) + ".", pl = p + "mix.left.", pr = p + "mix.right.", pm = p + "mlp.";
        auto rows = [&](const std::string& name, int first, int n) { T.matrix(name, (char*)L.wmix + (size_t)first * D * es, n, D, D); };
        rows(pl + "q", L.proj.lq, a.heads * a.dim); rows(pl + "k", L.proj.lk, a.kv_heads * a.dim); rows(pl + "v", L.proj.lv, a.kv_heads * a.vdim);
        rows(pl + "g", L.proj.lg, a.heads);
        rows(pr + "q", L.proj.rq, r.heads * r.dim); rows(pr + "k", L.proj.rk, r.heads * r.dim); rows(pr + "v", L.proj.rv, r.heads * r.vdim);
        rows(pr + "g", L.proj.rg, r.heads * r.vdim); rows(pr + "i", L.proj.ri, r.heads); rows(pr + "f", L.proj.rf, r.heads);
        T.matrix(pl + "o", L.wo_l, D, a.heads * a.vdim, L.kl);
        T.matrix(pr + "o", L.wo_r, D, r.heads * r.vdim, L.kr);
        T.vector(pl + "q.norm", L.q_norm, a.heads * a.dim, 0.f, 1.f); T.vector(pl + "k.norm", L.k_norm, a.kv_heads * a.dim, 0.f, 1.f);
        T.vector(pl + "sink", L.sink, a.heads, 0.f, 0.f);
        T.vector(pl + "out", L.out_l, D, 0.f, 1.f); T.vector(pr + "out", L.out_r, D, 0.f, 1.f);
        T.vector(pr + "norm", L.mem_norm, r.heads * r.vdim, 0.f, 1.f);
        T.vector(pr + "i.b", L.ib, r.heads, 0.f, 0.f); T.vector(pr + "f.b", L.fb, r.heads, 0.f, 3.f);
        T.vector(p + "norm1", L.gain1, D, 1.f, 0.f);
        {   // distance-bias slopes 2^(-8 (h + 1) / H)
            std::vector<float> sl(a.heads);
            for (int i = 0; i < a.heads; ++i) sl[i] = (float)std::pow(2.0, -8.0 * (i + 1) / a.heads);
            if (!T.rc && cudaMemcpy(L.slopes, sl.data(), sl.size() * 4, cudaMemcpyHostToDevice) != cudaSuccess) T.rc = fail(m, CD_ERR_CUDA, "upload of the distance-bias slopes");
        }
        if (f.kind == FfnCfg::NONE) continue;
        T.vector(p + "norm2", L.gain2, D, 1.f, 0.f);
        auto ffn = [&](const std::string& q, size_t i) {
            char* w13 = (char*)L.w13 + i * 2 * L.ffp * D * es;
            T.matrix(q + "gate", w13, f.ff, D, D, 2, 0);
            T.matrix(q + "up", w13, f.ff, D, D, 2, 1);
            T.matrix(q + "down", (char*)L.w2 + i * D * L.ffp * es, D, f.ff, L.ffp);
        };
        if (f.kind == FfnCfg::DENSE) {
            ffn(pm, 0);
        } else {
            T.matrix(pm + "router", L.wr, f.experts, D, D);
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
