// The dense decoder family: weights, per-token step (one persistent kernel, or one kernel per operator), construction
// from host tensors or the synthetic generator, and cache seeding.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <type_traits>

#include "step.cuh"
#include "mega.cuh"

using namespace cd;

namespace {
template <typename KT, int HD>
cudaError_t launch_attn_hd(cd_model* m, const cd_layer_dev& L) {
    const cd_config& c = m->cfg;
    const float scale = 1.0f / std::sqrt((float)c.hd);  // ATTN_SCALE, lib.rs:1352
    cudaLaunchConfig_t lc = {};
    lc.gridDim = dim3(c.heads, m->nsplit);
    lc.blockDim = dim3(128);
    lc.stream = m->stream;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = 1;
    lc.attrs = at;
    lc.numAttrs = m->pdl ? 1 : 0;
    cudaError_t e = cudaLaunchKernelEx(&lc, attn_decode_kernel<KT, HD>, (const float*)m->q, (const KT*)L.kv, (const int*)m->page_table,
                                       (const DevState*)m->st, m->part_acc, m->part_ml, m->counters, m->attn, c.kv_heads,
                                       c.gqa_ratio, m->page_tokens, m->nsplit, scale);
    count_launch(m);
    return e;
}

template <typename KT>
cudaError_t launch_attn(cd_model* m, const cd_layer_dev& L) {
    return m->cfg.hd == 128 ? launch_attn_hd<KT, 128>(m, L) : launch_attn_hd<KT, 64>(m, L);
}

// ------------------------------------------------------------------ persistent kernel launch
template <typename WT, typename KT, int ND, int NH, bool TPAR>
cudaError_t launch_mega_t(cd_model* m, int input_embed, int want_logits) {
    constexpr int RD = ND == 1 ? 4 : ND == 2 ? 2 : 1;
    constexpr int RH = NH == 1 ? 4 : NH == 2 ? 2 : 1;
    const cd_config& c = m->cfg;
    auto kern = decode_mega_kernel<WT, KT, ND, RD, NH, RH, TPAR>;
    const int grid = m->sm_count;
    const size_t es = sizeof(WT);
    const size_t stage_cap = (std::max((size_t)RD * c.dim * es, (size_t)RH * c.hidden * es) + 127) / 128 * 128;
    int max_rows = 0;
    for (int n : {c.q_dim + 2 * c.kv_dim, c.dim, 2 * c.hidden, want_logits ? m->v_loc : 0}) max_rows = std::max(max_rows, n / grid + 2);
    const int xs_dim = m->tp_world > 1 ? std::max(c.q_dim, c.dim) : c.q_dim;
    const size_t fixed = ((size_t)max_rows * (GEMV_CONSUMERS / 32) + 32 * MEGA_GROUPS + mega_attn_smem_floats(xs_dim)) * sizeof(float) + 32 +
                         (size_t)((m->pages_per_seq + 3) & ~3) * 4 + 2 * 16 * 8 + 128;
    const size_t budget = (size_t)m->ring_kb * 1024;
    if (fixed + 2 * stage_cap > budget) return cudaErrorInvalidConfiguration;
    const int nstages = (int)std::min<size_t>(16, (budget - fixed) / stage_cap) & ~1;  // even: slots alternate between the two consumer groups
    const size_t smem = (size_t)nstages * stage_cap + fixed;
    // attention tiles: the largest power-of-two run of cached positions that stays inside a page and fits a stage
    int tile = 64;
    while (tile > 1 && (tile > m->page_tokens || m->page_tokens % tile || (size_t)tile * c.hd * sizeof(KT) > stage_cap)) tile >>= 1;
    static size_t smem_set = 0;
    if (smem > smem_set) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        smem_set = smem;
    }
    MegaParams p;
    p.layers = (const MegaLayer*)m->mega_layers;
    p.embed = m->embed; p.lm_head = m->lm_head; p.gamma_final = m->gamma_final;
    p.x_a = m->x_a; p.x_b = m->x_b; p.q = m->q; p.gate = m->gate; p.logits = m->logits; p.norm_final = m->norm_final;
    p.part_acc = m->part_acc; p.part_ml = m->part_ml; p.grid_counter = m->grid_counter;
    p.st = m->st; p.page_table = m->page_table; p.rope = m->rope;
    p.dim = c.dim; p.hidden = c.hidden; p.heads = c.heads; p.kv_heads = c.kv_heads; p.hd = c.hd; p.nlayers = c.nlayers;
    p.vocab = m->v_loc; p.embed_rows = m->full_cfg.vocab; p.q_dim = c.q_dim; p.kv_dim = c.kv_dim; p.gqa = c.gqa_ratio; p.page_tokens = m->page_tokens;
    p.activation = m->opt.activation; p.alpha = m->alpha; p.attn_scale = 1.0f / std::sqrt((float)c.hd);
    p.trace = m->mega_trace;
    p.npages = m->pages_per_seq;
    p.tile_tokens = tile;
    p.wait_ns = m->wait_ns;
    p.tp = m->tp;  // world <= 1 on one GPU
    p.tp.wait_ns = m->wait_ns;
    p.xs_dim = xs_dim;
    p.nstages = nstages; p.stage_cap = (uint32_t)stage_cap; p.rows_cap = max_rows; p.input_embed = input_embed; p.want_logits = want_logits;
    cudaLaunchConfig_t lc = {};
    lc.gridDim = dim3(grid);
    lc.blockDim = dim3(MEGA_THREADS);
    lc.dynamicSmemBytes = smem;
    lc.stream = m->stream;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeCooperative;  // all CTAs resident: they meet at grid barriers
    at[0].val.cooperative = 1;
    lc.attrs = at;
    lc.numAttrs = 1;
    cudaError_t e = cudaLaunchKernelEx(&lc, kern, p);
    count_launch(m);
    return e;
}

template <typename WT, typename KT, bool TPAR>
cudaError_t launch_mega_tp(cd_model* m, int input_embed, int want_logits) {
    switch (m->mega_nd * 10 + m->mega_nh) {
        case 11: return launch_mega_t<WT, KT, 1, 1, TPAR>(m, input_embed, want_logits);
        case 12: return launch_mega_t<WT, KT, 1, 2, TPAR>(m, input_embed, want_logits);
        case 24: return launch_mega_t<WT, KT, 2, 4, TPAR>(m, input_embed, want_logits);
        case 26: return launch_mega_t<WT, KT, 2, 6, TPAR>(m, input_embed, want_logits);
        default: return cudaErrorInvalidConfiguration;
    }
}
template <typename WT, typename KT>
cudaError_t launch_mega(cd_model* m, int input_embed, int want_logits) {
    if constexpr (!std::is_same<WT, float>::value) {  // the tensor-parallel form exists for the 16-bit storage types
        if (m->tp_world > 1) return launch_mega_tp<WT, KT, true>(m, input_embed, want_logits);
    }
    return launch_mega_tp<WT, KT, false>(m, input_embed, want_logits);
}

// One token through the whole model; everything is enqueued on m->stream.
// WT: storage of the embedding and the LM head; LT: row format of the linears; KT: storage of the KV cache.
template <typename WT, typename LT, typename KT>
cudaError_t enqueue_step_t(cd_model* m, const cd_step& p) {
    const cd_config& c = m->cfg;
    cudaError_t e;
#define TRY(x) do { e = (x); if (e != cudaSuccess) return e; } while (0)
    m->cur_cls = CLS_MISC;
    if (p.input == 2) {
        next_prompt_kernel<<<1, 1, 0, m->stream>>>(m->st, m->prompt_dev);
        count_launch(m);
    }
    const bool use_mega = std::is_same<WT, LT>::value && m->mega && m->mega_nd > 0 && !m->profiling;
    if (use_mega) {
        if constexpr (std::is_same<WT, LT>::value) TRY((launch_mega<WT, KT>(m, p.input >= 1 ? 1 : 0, p.head != HEAD_NONE ? 1 : 0)));
    } else if (p.input >= 1) {
        embed_kernel<WT><<<std::max(1, c.dim / 256), 256, 0, m->stream>>>((const WT*)m->embed, m->st, m->x_a, c.dim, m->full_cfg.vocab);
        count_launch(m);
        TRY(cudaGetLastError());
    }
    for (int l = 0; l < c.nlayers && !use_mega; ++l) {
        const cd_layer_dev& L = m->layers[l];
        EpiQKV<KT> eq{m->q, (KT*)L.kv, m->page_table, m->st, m->rope, c.q_dim, c.kv_dim, c.hd, c.kv_heads, m->page_tokens};
        const bool last = l + 1 == c.nlayers;
        auto hint = [&](const void* w, int K, int N, int unit, bool head = false) {
            const uint32_t rb = head ? (uint32_t)(K * sizeof(WT)) : Wfmt<LT>::row_stride(K);
            m->next_stream = NextStream{m->prefetch_kb > 0 ? w : nullptr, rb, N / unit, unit, (uint32_t)m->prefetch_kb * 1024u};
        };
        const bool tp_on = m->tp_world > 1;
        EpiPush push{m->tp};
        m->cur_cls = CLS_QKV;
        hint(L.wo, c.q_dim, c.dim, 1);
        if (tp_on && l > 0) { m->tp_in.in_reduce = 2 * l; m->tp_in.res = m->x_b; m->tp_in.x_out = m->x_a; }  // x = x2 + alpha * sum(W2 partials)
        TRY((launch_gemv<LT, 2, true>(m, L.wqkv, m->x_a, L.gamma1, nullptr, c.q_dim + 2 * c.kv_dim, c.dim, eq)));
        m->cur_cls = CLS_ATTN;
        TRY(launch_attn<KT>(m, L));
        m->cur_cls = CLS_WO;
        hint(L.w13, c.dim, 2 * c.hidden, 2);
        push.tp.ar_out = 2 * l + 1;
        if (tp_on) TRY((launch_gemv<LT, 1, false>(m, L.wo, m->attn, nullptr, nullptr, c.dim, c.q_dim, push)));
        else TRY((launch_gemv<LT, 1, false>(m, L.wo, m->attn, nullptr, nullptr, c.dim, c.q_dim, EpiResidual{m->x_a, m->x_b, m->alpha})));
        m->cur_cls = CLS_W13;
        hint(L.w2, c.hidden, c.dim, 1);
        if (tp_on) { m->tp_in.in_reduce = 2 * l + 1; m->tp_in.res = m->x_a; m->tp_in.x_out = m->x_b; }  // x2 = x + alpha * sum(Wo partials)
        TRY((launch_gemv<LT, 2, true>(m, L.w13, m->x_b, L.gamma2, nullptr, 2 * c.hidden, c.dim, EpiGate{m->gate, m->opt.activation})));
        m->cur_cls = CLS_W2;
        if (!last) hint(m->layers[l + 1].wqkv, c.dim, c.q_dim + 2 * c.kv_dim, 2);
        else if (p.head != HEAD_NONE) hint(m->lm_head, c.dim, m->v_loc, 1, true);
        else hint(m->layers[0].wqkv, c.dim, c.q_dim + 2 * c.kv_dim, 2);
        push.tp.ar_out = 2 * l + 2;
        if (tp_on) TRY((launch_gemv<LT, 1, false>(m, L.w2, m->gate, nullptr, nullptr, c.dim, c.hidden, push)));
        else TRY((launch_gemv<LT, 1, false>(m, L.w2, m->gate, nullptr, nullptr, c.dim, c.hidden, EpiResidual{m->x_b, m->x_a, m->alpha})));
    }
    return enqueue_head_t<WT, LT>(m, p, use_mega, m->tp_world > 1 ? 2u * (unsigned int)c.nlayers : 0u, 2 * c.nlayers);
#undef TRY
}

cudaError_t dense_step(cd_model* m, const cd_step& p) {
    const bool kv16 = m->kv_dtype == CD_DTYPE_F16;  // otherwise the cache has the embedding's type (resolve_kv_dtype admits nothing else)
    switch (m->opt.weight_dtype) {
        case CD_DTYPE_F32: return enqueue_step_t<float, float, float>(m, p);
        case CD_DTYPE_F16: return enqueue_step_t<__half, __half, __half>(m, p);
        case CD_DTYPE_FP8_E4M3: return kv16 ? enqueue_step_t<__nv_bfloat16, Fp8Row, __half>(m, p) : enqueue_step_t<__nv_bfloat16, Fp8Row, __nv_bfloat16>(m, p);
        case CD_DTYPE_INT4_G32: return kv16 ? enqueue_step_t<__nv_bfloat16, Int4G32, __half>(m, p) : enqueue_step_t<__nv_bfloat16, Int4G32, __nv_bfloat16>(m, p);
        default: return kv16 ? enqueue_step_t<__nv_bfloat16, __nv_bfloat16, __half>(m, p) : enqueue_step_t<__nv_bfloat16, __nv_bfloat16, __nv_bfloat16>(m, p);
    }
}

cudaError_t dense_head_only(cd_model* m) {
    cudaError_t e = cudaSuccess;
    DISPATCH_WT(EMBED_DTYPE(m), WT, e = enqueue_head_only_t<WT>(m));
    return e;
}

const cd_family DENSE_FAMILY = {"dense", dense_step, dense_head_only, prefill_batched, prefill_hidden_row, decode_samples, prefill_release, nullptr, nullptr, nullptr};

}  // namespace

namespace cd {

static int validate(const cd_config& c, int dtype) {
    if (c.dim <= 0 || c.hidden <= 0 || c.heads <= 0 || c.kv_heads <= 0 || c.hd <= 0 || c.seq <= 0 || c.nlayers <= 0 || c.vocab <= 0)
        return fail(nullptr, CD_ERR_INVALID, "config contains a non-positive dimension");
    if (c.q_dim != c.heads * c.hd || c.kv_dim != c.kv_heads * c.hd || c.heads % c.kv_heads != 0 || c.gqa_ratio != c.heads / c.kv_heads)
        return fail(nullptr, CD_ERR_INVALID, "q_dim / kv_dim / gqa_ratio inconsistent with heads, kv_heads and hd");
    if (c.hd != 64 && c.hd != 128) return fail(nullptr, CD_ERR_UNSUPPORTED, "head dimension must be 64 or 128");
    if (dtype < CD_DTYPE_F32 || dtype > CD_DTYPE_INT4_G32) return fail(nullptr, CD_ERR_INVALID, "unknown weight dtype");
    const int epc = dtype == CD_DTYPE_F32 ? 4 : dtype == CD_DTYPE_FP8_E4M3 ? 16 : dtype == CD_DTYPE_INT4_G32 ? 32 : 8;
    const int kmax = dtype >= CD_DTYPE_FP8_E4M3 ? 4 * 256 * 16 : 8 * 256 * epc;
    if (c.dim % 8 || c.q_dim % 8 || c.hidden % 8) return fail(nullptr, CD_ERR_UNSUPPORTED, "dim, q_dim and hidden must be multiples of 8");
    if (c.dim % epc || c.q_dim % epc || c.hidden % epc) return fail(nullptr, CD_ERR_UNSUPPORTED, "dim, q_dim and hidden must be multiples of the quantisation chunk (16 for FP8, 32 for INT4)");
    if (c.dim > kmax || c.q_dim > kmax || c.hidden > kmax) return fail(nullptr, CD_ERR_UNSUPPORTED, "inner dimension too large for the GEMV tiling");
    return CD_OK;
}

int dense_alloc(const cd_config* cfg, const cd_options* opts_in, int untied, cd_model** out) {
    *out = nullptr;
    cd_options opts;
    memset(&opts, 0, sizeof(opts));
    opts.device = -1;
    if (opts_in) opts = *opts_in;
    int rc = validate(*cfg, opts.weight_dtype);
    if (rc) return rc;
    const int tpw = std::max(1, (int)opts.tp_world), tpr = tpw > 1 ? (int)opts.tp_rank : 0;
    AllocSpec spec;
    spec.family = &DENSE_FAMILY;
    spec.local = *cfg;
    if (tpw > 1) {
        cd_config& local = spec.local;
        if (opts.weight_dtype == CD_DTYPE_INT4_G32 && ((cfg->q_dim / tpw) % 32 || (cfg->hidden / tpw) % 32))
            return fail(nullptr, CD_ERR_UNSUPPORTED, "INT4 groups of 32 must not straddle tensor-parallel shards (q_dim/world and hidden/world multiples of 32)");
        if (tpw > TP_MAX || tpr < 0 || tpr >= tpw) return fail(nullptr, CD_ERR_INVALID, "tensor-parallel rank / world out of range");
        if (cfg->kv_heads % tpw || cfg->heads % tpw || cfg->hidden % (8 * tpw))
            return fail(nullptr, CD_ERR_UNSUPPORTED, "heads, kv_heads and hidden/8 must be divisible by the tensor-parallel world size");
        local.heads /= tpw; local.kv_heads /= tpw; local.hidden /= tpw; local.q_dim /= tpw; local.kv_dim /= tpw;
        if ((rc = validate(local, opts.weight_dtype))) return rc;
        spec.sharded_head = true;
        // 16-bit models also run the prompt as GEMMs: two buffers of partial sums for up to seq prompt rows
        if (opts.weight_dtype == CD_DTYPE_BF16 || opts.weight_dtype == CD_DTYPE_F16) spec.tp_prefill_rows = ((size_t)cfg->seq + 127) / 128 * 128;
    }
    const cd_config c = spec.local;
    spec.kv_row_elems.assign(c.nlayers, (size_t)2 * c.kv_heads * c.hd);  // K and V of every kv head
    spec.rope_dim = c.hd;
    spec.attn_parts = MEGA_MAX_PARTS;  // CTAs of the persistent kernel that share a head
    const size_t ml_bytes = align_up((size_t)c.nlayers * sizeof(MegaLayer), 256);
    spec.family_ws_bytes = ml_bytes + (size_t)2 * (10 * c.nlayers + 2) * 8;
    cd_model* m = nullptr;
    if ((rc = model_alloc(cfg, opts, untied, spec, &m))) return rc;
    auto bail = [&](int code) { cd_model_destroy(m); return code; };
#define CKB(call) do { cudaError_t e_ = (call); if (e_ != cudaSuccess) { fail(nullptr, CD_ERR_CUDA, std::string(#call) + ": " + cudaGetErrorString(e_)); return bail(CD_ERR_CUDA); } } while (0)
    const size_t D = c.dim, Q = c.q_dim, KV = c.kv_dim, H = c.hidden;
    const int dt = opts.weight_dtype;
    size_t off = 0;
    auto carve = [&](size_t bytes) { size_t o = off; off = align_up(off + bytes, 256); return o; };
    struct LO { size_t wqkv, wo, w13, w2, g1, g2; };
    std::vector<LO> lo(c.nlayers);
    for (auto& l : lo) {
        l.wqkv = carve((Q + 2 * KV) * lin_row_bytes(dt, c.dim)); l.wo = carve(D * lin_row_bytes(dt, c.q_dim)); l.w13 = carve(2 * H * lin_row_bytes(dt, c.dim));
        l.w2 = carve(D * lin_row_bytes(dt, c.hidden)); l.g1 = carve(D * 4); l.g2 = carve(D * 4);
    }
    CKB(cudaMalloc(&m->layer_arena, off));
    m->weight_bytes += off;
    char* wb = (char*)m->layer_arena;
    for (int l = 0; l < c.nlayers; ++l) {
        m->layers[l].wqkv = wb + lo[l].wqkv; m->layers[l].wo = wb + lo[l].wo; m->layers[l].w13 = wb + lo[l].w13;
        m->layers[l].w2 = wb + lo[l].w2; m->layers[l].gamma1 = (float*)(wb + lo[l].g1); m->layers[l].gamma2 = (float*)(wb + lo[l].g2);
    }
    {   // gammas default to 1 (LayerWeights::random, layer.rs:711-712)
        std::vector<float> ones(D, 1.0f);
        for (auto& L : m->layers) {
            CKB(cudaMemcpy(L.gamma1, ones.data(), D * 4, cudaMemcpyHostToDevice));
            CKB(cudaMemcpy(L.gamma2, ones.data(), D * 4, cudaMemcpyHostToDevice));
        }
    }
    {   // per-layer pointer table and tiling of the persistent kernel
        m->mega_layers = m->family_ws;
        if (opts.test_flags & 4) m->mega_trace = (unsigned long long*)(m->family_ws + ml_bytes);  // test_flags bit 2: phase stamps of the persistent kernel
        std::vector<MegaLayer> ml(c.nlayers);
        for (int l = 0; l < c.nlayers; ++l) {
            const cd_layer_dev& L = m->layers[l];
            ml[l] = MegaLayer{L.wqkv, L.wo, L.w13, L.w2, L.gamma1, L.gamma2, L.kv};
        }
        CKB(cudaMemcpyAsync(m->mega_layers, ml.data(), ml.size() * sizeof(MegaLayer), cudaMemcpyHostToDevice, m->stream));
        CKB(cudaStreamSynchronize(m->stream));
        const int epc = dt == CD_DTYPE_F32 ? 4 : 8;
        const int nd = (c.dim / epc + 255) / 256, nh = (c.hidden / epc + 255) / 256;
        // (c is this rank's shard under tensor parallelism: hidden and q_dim shrink, dim does not)
        const bool combo = (nd == 1 && (nh == 1 || nh == 2)) || (nd == 2 && nh >= 3 && nh <= 6);
        if (combo && c.q_dim <= c.dim && c.gqa_ratio <= MEGA_MAX_GQA) { m->mega_nd = nd; m->mega_nh = nh == 3 ? 4 : nh == 5 ? 6 : nh; }
        // tensor parallel: measured on the 5B model, the persistent kernel wins at 2 ranks (601 against 569 tokens/s) and
        // loses at 8 (841 against 896), where a layer's data are 8 us and its fixed per-phase times dominate either way
        const bool mega_ok = !is_quant(dt) && (tpw == 1 || (tpw == 2 && dt != CD_DTYPE_F32));
        // one persistent kernel per token wherever its tiling covers the shape; test_flags bit 1 keeps one kernel per operator
        m->mega = (opts.test_flags & 2) == 0 && mega_ok && m->mega_nd > 0;
    }
#undef CKB
    *out = m;
    return CD_OK;
}

// where a reference tensor lands in the device layout
struct Placement {
    void* dst;
    int in, out, transposed, row_mul, row_off;
    bool vec;  // fp32 vector (gamma)
    int full_in, full_out, in0, out0;  // the shard's place inside the reference's full tensor
};

static int place(cd_model* m, int layer, int which, Placement* p) {
    const cd_config& c = m->cfg;        // local (sharded) sizes
    const cd_config& f = m->full_cfg;   // reference sizes
    const int r = m->tp_rank;
    const size_t rb = lin_row_bytes(m->opt.weight_dtype, c.dim);  // a row of wqkv
    if (which == T_EMBED) { *p = {m->embed, c.dim, f.vocab, 0, 1, 0, false, f.dim, f.vocab, 0, 0}; return CD_OK; }
    if (which == T_LM_HEAD) {
        if (!m->untied) return fail(m, CD_ERR_INVALID, "model has a tied head");
        *p = {m->lm_head, c.dim, m->v_loc, 0, 1, 0, false, f.dim, f.vocab, 0, m->v0};
        return CD_OK;
    }
    if (which == T_GAMMA_FINAL) { *p = {m->gamma_final, c.dim, 1, 0, 1, 0, true, c.dim, 1, 0, 0}; return CD_OK; }
    if (layer < 0 || layer >= c.nlayers) return fail(m, CD_ERR_INVALID, "layer index out of range");
    cd_layer_dev& L = m->layers[layer];
    switch (which) {  // heads and FFN columns are split across ranks; Wo and W2 are split along their input
        case T_WQ: *p = {L.wqkv, c.dim, c.q_dim, 1, 1, 0, false, f.dim, f.q_dim, 0, r * c.q_dim}; break;
        case T_WK: *p = {(char*)L.wqkv + (size_t)c.q_dim * rb, c.dim, c.kv_dim, 1, 1, 0, false, f.dim, f.kv_dim, 0, r * c.kv_dim}; break;
        case T_WV: *p = {(char*)L.wqkv + (size_t)(c.q_dim + c.kv_dim) * rb, c.dim, c.kv_dim, 1, 1, 0, false, f.dim, f.kv_dim, 0, r * c.kv_dim}; break;
        case T_WO: *p = {L.wo, c.q_dim, c.dim, 1, 1, 0, false, f.q_dim, f.dim, r * c.q_dim, 0}; break;
        case T_W1: *p = {L.w13, c.dim, c.hidden, 1, 2, 0, false, f.dim, f.hidden, 0, r * c.hidden}; break;
        case T_W3: *p = {L.w13, c.dim, c.hidden, 1, 2, 1, false, f.dim, f.hidden, 0, r * c.hidden}; break;
        case T_W2: *p = {L.w2, c.hidden, c.dim, 0, 1, 0, false, f.hidden, f.dim, r * c.hidden, 0}; break;  // already [out=dim, in=hidden]
        case T_GAMMA1: *p = {L.gamma1, c.dim, 1, 0, 1, 0, true, c.dim, 1, 0, 0}; break;
        case T_GAMMA2: *p = {L.gamma2, c.dim, 1, 0, 1, 0, true, c.dim, 1, 0, 0}; break;
        default: return fail(m, CD_ERR_INVALID, "unknown tensor id");
    }
    return CD_OK;
}

size_t model_tensor_elems(const cd_model* m, int which) {
    const cd_config& c = m->full_cfg;  // sizes of the tensors as stored in a checkpoint
    switch (which) {
        case T_EMBED: case T_LM_HEAD: return (size_t)c.vocab * c.dim;
        case T_GAMMA_FINAL: case T_GAMMA1: case T_GAMMA2: return c.dim;
        case T_WQ: case T_WO: return (size_t)c.dim * c.q_dim;
        case T_WK: case T_WV: return (size_t)c.dim * c.kv_dim;
        default: return (size_t)c.dim * c.hidden;
    }
}

static int ensure_staging(cd_model* m, size_t bytes) {
    if (m->staging_bytes >= bytes) return CD_OK;
    if (m->staging) cudaFree(m->staging);
    m->staging = nullptr; m->staging_bytes = 0;
    CK(m, cudaMalloc(&m->staging, bytes));
    m->staging_bytes = bytes;
    return CD_OK;
}

static int ensure_staging2(cd_model* m, size_t bytes) {
    if (m->staging2_bytes >= bytes) return CD_OK;
    if (m->staging2) cudaFree(m->staging2);
    m->staging2 = nullptr; m->staging2_bytes = 0;
    CK(m, cudaMalloc(&m->staging2, bytes));
    m->staging2_bytes = bytes;
    return CD_OK;
}

// staging2 holds this rank's output rows as [out, full_in] fp32 (whole rows, so that an input-split shard of
// Wo / W2 is quantised with the scales of the unsharded matrix); write columns in0 .. in0 + in - 1 to their
// place in the quantised row format
static int quantize_rows(cd_model* m, const Placement& p) {
    const int grid = std::min(p.out, m->sm_count * 8);
    if (m->opt.weight_dtype == CD_DTYPE_FP8_E4M3)
        quantize_fp8_rows_kernel<<<grid, 256, 0, m->stream>>>((const float*)m->staging2, (unsigned char*)p.dst, p.in, p.out, p.row_mul, p.row_off, p.full_in, p.in0);
    else
        quantize_int4_rows_kernel<<<grid, 256, 0, m->stream>>>((const float*)m->staging2, (unsigned char*)p.dst, p.in, p.out, p.row_mul, p.row_off, p.full_in, p.in0);
    CK(m, cudaGetLastError());
    CK(m, cudaStreamSynchronize(m->stream));
    return CD_OK;
}

int model_set_tensor_f32(cd_model* m, int layer, int which, const float* host) {
    Placement p;
    int rc = place(m, layer, which, &p);
    if (rc) return rc;
    if (!host) return fail(m, CD_ERR_INVALID, "null tensor pointer");
    if (p.vec) { CK(m, cudaMemcpy(p.dst, host, (size_t)p.in * 4, cudaMemcpyHostToDevice)); return CD_OK; }
    const size_t n = (size_t)p.full_in * p.full_out;  // the whole reference tensor is staged; the kernel picks the shard
    rc = ensure_staging(m, n * 4);
    if (rc) return rc;
    CK(m, cudaMemcpyAsync(m->staging, host, n * 4, cudaMemcpyHostToDevice, m->stream));
    const dim3 grid((p.in + 31) / 32, (p.out + 31) / 32), block(32, 8);
    if (is_quant(m->opt.weight_dtype) && which >= T_WQ && which <= T_W2) {
        // this rank's output rows, whole, in GEMV orientation as fp32 first, then quantised row by row
        rc = ensure_staging2(m, (size_t)p.full_in * p.out * 4);
        if (rc) return rc;
        const dim3 gridf((p.full_in + 31) / 32, (p.out + 31) / 32);
        relayout_kernel<float><<<gridf, block, 0, m->stream>>>((const float*)m->staging, (float*)m->staging2, p.full_in, p.out, p.transposed, 1, 0,
                                                               p.full_in, p.full_out, 0, p.out0);
        return quantize_rows(m, p);
    }
    DISPATCH_WT(m->opt.weight_dtype, WT,
                relayout_kernel<WT><<<grid, block, 0, m->stream>>>((const float*)m->staging, (WT*)p.dst, p.in, p.out, p.transposed, p.row_mul, p.row_off,
                                                                   p.full_in, p.full_out, p.in0, p.out0));
    CK(m, cudaGetLastError());
    CK(m, cudaStreamSynchronize(m->stream));
    return CD_OK;
}

// Bytes of one linear as a quantised checkpoint stores it: full_out rows in GEMV orientation, each in the device's row
// format for its whole input width (FP8: codes, fp32 row scale, padding; INT4: nibbles, fp16 group scales, padding).
size_t model_quant_tensor_bytes(const cd_model* m, int which) {
    const cd_config& f = m->full_cfg;
    int in, out;
    switch (which) {
        case T_WQ: in = f.dim; out = f.q_dim; break;
        case T_WK: case T_WV: in = f.dim; out = f.kv_dim; break;
        case T_WO: in = f.q_dim; out = f.dim; break;
        case T_W1: case T_W3: in = f.dim; out = f.hidden; break;
        case T_W2: in = f.hidden; out = f.dim; break;
        default: return 0;
    }
    return (size_t)out * lin_row_bytes(m->opt.weight_dtype, in);
}

// Upload one linear from stored quantised rows (the whole matrix, see model_quant_tensor_bytes): this rank's rows, and of
// an input-split matrix (Wo, W2) this rank's columns with the whole row's scale (FP8) or its own groups' scales (INT4) -
// byte for byte what quantising the fp32 tensor at load produces.
int model_set_quant_rows(cd_model* m, int layer, int which, const void* host) {
    if (!is_quant(m->opt.weight_dtype) || which < T_WQ || which > T_W2) return fail(m, CD_ERR_INVALID, "stored quantised rows exist for the linears of a quantised model only");
    Placement p;
    int rc = place(m, layer, which, &p);
    if (rc) return rc;
    if (!host) return fail(m, CD_ERR_INVALID, "null tensor pointer");
    const int dt = m->opt.weight_dtype;
    const size_t sf = lin_row_bytes(dt, p.full_in), sl = lin_row_bytes(dt, p.in);
    const char* src = (const char*)host + (size_t)p.out0 * sf;
    char* dst = (char*)p.dst + (size_t)p.row_off * sl;
    const size_t dpitch = (size_t)p.row_mul * sl;
    if (dt == CD_DTYPE_FP8_E4M3) {
        CK(m, cudaMemcpy2DAsync(dst, dpitch, src + p.in0, sf, (size_t)p.in, (size_t)p.out, cudaMemcpyHostToDevice, m->stream));
        CK(m, cudaMemcpy2DAsync(dst + p.in, dpitch, src + p.full_in, sf, sl - (size_t)p.in, (size_t)p.out, cudaMemcpyHostToDevice, m->stream));
    } else {
        const size_t nib = (size_t)p.in / 2, sc = (size_t)p.in / 16;  // bytes of nibbles, of fp16 scales (one per 32 inputs)
        CK(m, cudaMemcpy2DAsync(dst, dpitch, src + p.in0 / 2, sf, nib, (size_t)p.out, cudaMemcpyHostToDevice, m->stream));
        CK(m, cudaMemcpy2DAsync(dst + nib, dpitch, src + p.full_in / 2 + p.in0 / 16, sf, sc, (size_t)p.out, cudaMemcpyHostToDevice, m->stream));
        if (sl > nib + sc) CK(m, cudaMemset2DAsync(dst + nib + sc, dpitch, 0, sl - nib - sc, (size_t)p.out, m->stream));
    }
    CK(m, cudaStreamSynchronize(m->stream));
    return CD_OK;
}

// This rank's rows of one linear, in the device's row format for the local input width, to host memory.
int model_get_quant_rows(cd_model* m, int layer, int which, void* host, size_t cap) {
    if (!is_quant(m->opt.weight_dtype) || which < T_WQ || which > T_W2) return fail(m, CD_ERR_INVALID, "quantised rows exist for the linears of a quantised model only");
    Placement p;
    int rc = place(m, layer, which, &p);
    if (rc) return rc;
    const size_t sl = lin_row_bytes(m->opt.weight_dtype, p.in);
    if (!host || cap < (size_t)p.out * sl) return fail(m, CD_ERR_CAPACITY, "buffer too small for the tensor's rows");
    CK(m, cudaMemcpy2DAsync(host, sl, (const char*)p.dst + (size_t)p.row_off * sl, (size_t)p.row_mul * sl, sl, (size_t)p.out, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaStreamSynchronize(m->stream));
    return CD_OK;
}

// The embedding or the untied head (storage: 2 or 4 bytes per element) and the fp32 vectors, as stored on the device.
int model_get_plain(cd_model* m, int layer, int which, void* host, size_t cap) {
    Placement p;
    int rc = place(m, layer, which, &p);
    if (rc) return rc;
    if (!p.vec && which != T_EMBED && which != T_LM_HEAD) return fail(m, CD_ERR_INVALID, "not a plain tensor");
    const size_t bytes = p.vec ? (size_t)p.in * 4 : (size_t)p.in * p.out * esize(m->opt.weight_dtype);
    if (!host || cap < bytes) return fail(m, CD_ERR_CAPACITY, "buffer too small for the tensor");
    CK(m, cudaMemcpyAsync(host, p.dst, bytes, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaStreamSynchronize(m->stream));
    return CD_OK;
}

int model_set_tensor_synth(cd_model* m, int layer, int which, uint64_t seed, float std) {
    Placement p;
    int rc = place(m, layer, which, &p);
    if (rc) return rc;
    if (p.vec) return fail(m, CD_ERR_INVALID, "gammas are not synthesised");
    uint64_t uid = which == T_EMBED ? 0 : which == T_LM_HEAD ? 2 : synth_uid_layer(layer, which - T_WQ);
    const uint64_t key = synth_key(seed, uid);
    const float scale = std / 65536.0f;
    if (is_quant(m->opt.weight_dtype) && which >= T_WQ && which <= T_W2) {
        rc = ensure_staging2(m, (size_t)p.full_in * p.out * 4);
        if (rc) return rc;
        synth_kernel<float><<<m->sm_count * 8, 256, 0, m->stream>>>((float*)m->staging2, p.full_in, p.out, p.transposed, 1, 0, key, scale,
                                                                    p.full_in, p.full_out, 0, p.out0);
        return quantize_rows(m, p);
    }
    DISPATCH_WT(m->opt.weight_dtype, WT,
                synth_kernel<WT><<<m->sm_count * 8, 256, 0, m->stream>>>((WT*)p.dst, p.in, p.out, p.transposed, p.row_mul, p.row_off, key, scale,
                                                                      p.full_in, p.full_out, p.in0, p.out0));
    CK(m, cudaGetLastError());
    return CD_OK;
}

}  // namespace cd

extern "C" {

int cd_model_create(const cd_config* cfg, const cd_layer_init* layers, int nlayers, const cd_head_init* head,
                    const cd_options* opts, cd_model** out) {
    if (!cfg || !layers || !head || !out) return fail(nullptr, CD_ERR_INVALID, "null argument");
    *out = nullptr;
    if (nlayers != cfg->nlayers) return fail(nullptr, CD_ERR_INVALID, "layer count does not match cfg.nlayers");  // lib.rs:184
    cd_model* m = nullptr;
    int rc = dense_alloc(cfg, opts, head->lm_head != nullptr, &m);
    if (rc) return rc;
    auto set = [&](int l, int which, const float* p) { if (rc == CD_OK) rc = model_set_tensor_f32(m, l, which, p); };
    set(0, T_EMBED, head->embed);
    set(0, T_GAMMA_FINAL, head->gamma_final);
    if (head->lm_head) set(0, T_LM_HEAD, head->lm_head);
    for (int l = 0; l < nlayers; ++l) {
        const cd_layer_init& L = layers[l];
        set(l, T_WQ, L.wq); set(l, T_WK, L.wk); set(l, T_WV, L.wv); set(l, T_WO, L.wo);
        set(l, T_W1, L.w1); set(l, T_W3, L.w3); set(l, T_W2, L.w2); set(l, T_GAMMA1, L.gamma1); set(l, T_GAMMA2, L.gamma2);
    }
    if (rc == CD_OK) rc = model_finish(m);
    if (rc) { set_global_error(m->err); cd_model_destroy(m); return rc; }
    *out = m;
    return CD_OK;
}

int cd_model_create_synthetic(const cd_config* cfg, const cd_options* opts, uint64_t seed, float std, int untied_head,
                              cd_model** out) {
    if (!cfg || !out) return fail(nullptr, CD_ERR_INVALID, "null argument");
    *out = nullptr;
    cd_model* m = nullptr;
    int rc = dense_alloc(cfg, opts, untied_head != 0, &m);
    if (rc) return rc;
    auto syn = [&](int l, int which) { if (rc == CD_OK) rc = model_set_tensor_synth(m, l, which, seed, std); };
    syn(0, T_EMBED);
    if (untied_head) syn(0, T_LM_HEAD);
    for (int l = 0; l < cfg->nlayers; ++l)
        for (int w = T_WQ; w <= T_W2; ++w) syn(l, w);
    if (rc == CD_OK) rc = model_finish(m);
    if (rc) { set_global_error(m->err); cd_model_destroy(m); return rc; }
    *out = m;
    return CD_OK;
}

int cd_seed_layer_cache_cf(cd_model* m, int layer, size_t live_len, const float* k_cf, const float* v_cf) {
    if (!m || !k_cf || !v_cf) return fail(m, CD_ERR_INVALID, "null argument");
    if (m->family != &DENSE_FAMILY) return fail(m, CD_ERR_UNSUPPORTED, "only the dense family's cache can be seeded from K and V");
    if (m->tp_world > 1) return fail(m, CD_ERR_UNSUPPORTED, "not available on a tensor-parallel model: use the greedy entry points");
    const cd_config& c = m->cfg;
    if (layer < 0 || layer >= c.nlayers) return fail(m, CD_ERR_INVALID, "layer index out of range");
    live_len = std::min(live_len, (size_t)c.seq);
    const size_t n = (size_t)c.kv_dim * c.seq;
    int rc = ensure_staging(m, 2 * n * 4);
    if (rc) return rc;
    float* sk = (float*)m->staging;
    float* sv = sk + n;
    CK(m, cudaMemcpyAsync(sk, k_cf, n * 4, cudaMemcpyHostToDevice, m->stream));
    CK(m, cudaMemcpyAsync(sv, v_cf, n * 4, cudaMemcpyHostToDevice, m->stream));
    DISPATCH_WT(m->kv_dtype, KT,
                seed_kv_kernel<KT><<<m->sm_count * 4, 256, 0, m->stream>>>(sk, sv, (KT*)m->layers[layer].kv, m->page_table, c.seq,
                                                                           (int)live_len, c.kv_heads, c.hd, m->page_tokens));
    count_launch(m);
    CK(m, cudaGetLastError());
    CK(m, cudaStreamSynchronize(m->stream));
    return CD_OK;
}

}  // extern "C"
