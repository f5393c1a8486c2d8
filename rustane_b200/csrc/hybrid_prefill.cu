// Batched prompt pass of the configured decoder (hybrid.h): the linears as tensor-core GEMMs (prefill.cuh), the mixers,
// norms and routing over all rows (mixers_prefill.cuh).  Long prompts go through in pieces of a few thousand rows.
// bf16 models; others feed the prompt one token at a time.
#include "pf_launch.cuh"

#include <algorithm>
#include <cmath>
#include <cstdlib>
#include <cstring>

#include "hybrid.h"
#include "mixers_prefill.cuh"

namespace cd {
namespace {

constexpr size_t PIECE_ROWS = 4096;  // rows of the workspace at most (CD_PREFILL_ROWS overrides)

struct HybridPrefill {
    EncodeTiledFn encode = nullptr;
    size_t x_rows = 0, rows = 0;   // capacity: residual rows (the whole prompt), rows of one piece
    float* x = nullptr;            // [x_rows][width]
    void* arena = nullptr;
    // one piece
    float *proj = nullptr, *mem = nullptr, *raw = nullptr, *y = nullptr, *U = nullptr, *UN = nullptr, *gm = nullptr, *m_live = nullptr, *m_start = nullptr, *logits = nullptr,
          *sel_w = nullptr, *yp = nullptr;
    __nv_bfloat16 *xn = nullptr, *attn = nullptr, *memn = nullptr, *gate = nullptr, *perm = nullptr, *side = nullptr, *latent = nullptr;
    void *q = nullptr, *expanded = nullptr;
    int* zero_page = nullptr;      // the expanded keys' page table: one page
    size_t seen = 0;               // positions a latent layer expands for one piece at most
    int *sel_ids = nullptr, *slots = nullptr, *tile_group = nullptr;
    int max_tiles = 0;
    size_t perm_rows = 0;
};

struct Gemm {
    cd_model* m;
    HybridPrefill* w;
    bool split;
    cudaError_t e = cudaSuccess;
    const char* what = "";

    bool ok() const { return e == cudaSuccess; }
    // C[M][N] = A[M][K] (head and, under split, remainder) * B[rows][K]^T through `epi`
    template <class Epi>
    void operator()(const char* name, const __nv_bfloat16* hi, const __nv_bfloat16* lo, const void* B, int M, int N, int K, size_t b_rows, const Epi& epi,
                    const int* tile_group = nullptr, int group_rows = 0, size_t a_rows = 0) {
        if (!ok()) return;
        what = name;
        PfGemm p = {};
        p.M = M; p.N = N; p.K = K; p.b_zdiv = 1; p.page_tokens = m->page_tokens; p.err = &m->st->error;
        p.tile_group = tile_group; p.group_rows = group_rows;
        // tiles of 256 columns, of 128 where the wide ones would leave SMs without work
        const int mt = (M + PF_BM - 1) / PF_BM;
        const bool wide = (long)mt * ((N + 255) / 256) >= m->sm_count;
        CUtensorMap a[2], b;
        const CUtensorMapDataType dt = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
        if (!a_rows) a_rows = (size_t)mt * PF_BM;
        const bool maps = encode_2d(w->encode, &a[0], dt, hi, K, a_rows, (uint64_t)K * 2, PF_BM) && encode_2d(w->encode, &a[1], dt, split ? lo : hi, K, a_rows, (uint64_t)K * 2, PF_BM) &&
                          encode_2d(w->encode, &b, dt, B, K, b_rows, (uint64_t)K * 2, wide ? 256 : 128);
        if (!maps) { e = cudaErrorInvalidValue; return; }
        e = wide ? pf_launch<256>(m, split, a, b, p, true, 1, epi) : pf_launch<128>(m, split, a, b, p, true, 1, epi);
    }
};

template <typename KT>
cudaError_t launch_attn_window(cd_model* m, const AttnWindow& p, const KT* q_hi, const KT* q_lo, const KT* pool, __nv_bfloat16* hi, __nv_bfloat16* lo) {
    const size_t smem = attn_window_smem(p.a.kp, p.a.vp);
    const dim3 grid((p.rows + AW_TILE - 1) / AW_TILE, p.a.H * p.a.maps);
    auto go = [&](auto kern) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        kern<<<grid, 128, smem, m->stream>>>(p, q_hi, q_lo, pool, hi, lo);
        m->launches++;
        return cudaGetLastError();
    };
    if (p.a.vp <= 64) return go(attn_window_kernel<KT, __nv_bfloat16, 64>);
    if (p.a.vp <= 128) return go(attn_window_kernel<KT, __nv_bfloat16, 128>);
    return go(attn_window_kernel<KT, __nv_bfloat16, 256>);
}

// the buffer a latent layer's keys and values are expanded into: one page of `positions`
AttnDims expanded_dims(const cd_hybrid_layer& L, int positions) {
    const MlaDims& d = L.ld;
    const int k = d.nope_n + d.rope_n;
    return AttnDims{d.heads, d.heads, k, d.vdim, pad_to(k, 16), pad_to(d.vdim, 16), 1, d.window, positions, L.cfg.latent.scale, d.eps, 0.0f, 1, 0, 0.0f, 1.0f, Rotation{}};
}

int ensure_workspace(cd_model* m, HybridPrefill* w, size_t n, size_t piece) {
    const cd_hybrid_state& S = *m->hybrid;
    const size_t D = m->cfg.dim;
    auto cuda_fail = [&](cudaError_t e) { return fail(m, CD_ERR_CUDA, std::string("prompt-pass workspace: ") + cudaGetErrorString(e)); };
    const size_t x_rows = round_up(n, PF_BM);
    size_t rows = round_up(std::min(n, piece), PF_BM);
    if (x_rows > w->x_rows) {
        if (w->x) cudaFree(w->x);
        w->x = nullptr;
        w->x_rows = 0;
        const cudaError_t e = cudaMalloc((void**)&w->x, x_rows * D * 4);
        if (e != cudaSuccess) return cuda_fail(e);
        w->x_rows = x_rows;
    }
    // positions the new rows of a piece see, new ones included
    size_t seen = 0;
    for (const auto& L : S.layers)
        if (L.cfg.mixer == HybridLayerCfg::LATENT) seen = std::max(seen, L.ld.window > 0 ? std::min(rows + L.ld.window, m->len + n) : m->len + n);
    seen = round_up(seen, PF_BM);
    if (rows <= w->rows && seen <= w->seen) return CD_OK;
    rows = std::max(rows, w->rows);
    seen = std::max(seen, w->seen);
    if (w->arena) cudaFree(w->arena);
    w->arena = nullptr;
    w->rows = w->seen = 0;
    size_t raw = 0, lat = 0, exp = 0, proj = 0, mem = 0, kl = 0, kr = 0, gate = 0, q = 0, uf = 0, nf = 0, hm = 0, experts = 0, top = 0, moe_ff = 0;
    for (const auto& L : S.layers) {
        proj = std::max<size_t>(proj, L.proj.rows); mem = std::max<size_t>(mem, (size_t)L.md.H * L.md.vdim);
        kl = std::max<size_t>(kl, L.kl); kr = std::max<size_t>(kr, L.cfg.mixer == HybridLayerCfg::MEMORY ? L.kl : L.kr);
        q = std::max<size_t>(q, (size_t)L.ad.H * L.ad.kr());
        if (L.ad.maps > 1) raw = std::max<size_t>(raw, (size_t)L.ad.H * L.ad.maps * L.ad.vdim);
        if (L.cfg.mixer == HybridLayerCfg::LATENT) {
            const AttnDims x = expanded_dims(L, 1);
            q = std::max<size_t>(q, (size_t)x.H * x.kp); lat = std::max<size_t>(lat, L.ld.latent); exp = std::max<size_t>(exp, x.page_elems());
        }
        uf = std::max<size_t>(uf, L.md.s_floats()); nf = std::max<size_t>(nf, (size_t)L.md.H * L.md.dim); hm = std::max<size_t>(hm, L.md.H);
        const FfnCfg& f = L.cfg.mlp;
        if (f.kind == FfnCfg::DENSE) gate = std::max<size_t>(gate, L.ffp);
        if (f.kind == FfnCfg::MOE) {
            experts = std::max<size_t>(experts, f.experts); top = std::max<size_t>(top, f.top); moe_ff = std::max<size_t>(moe_ff, L.ffp);
        }
    }
    const size_t chunks = (rows + MEM_CHUNK - 1) / MEM_CHUNK, y_ld = round_up(D, 32);
    w->max_tiles = experts ? (int)(rows * top / PF_BM + experts) : 0;
    w->perm_rows = (size_t)w->max_tiles * PF_BM;
    size_t off = 0;
    std::vector<std::pair<void**, size_t>> places;
    auto carve = [&](void* p, size_t bytes) { places.push_back({(void**)p, off}); off = round_up(off + bytes, 256); };
    carve(&w->raw, rows * raw * 4); carve(&w->side, 2 * rows * S.side_pad() * 2);
    carve(&w->latent, 2 * seen * lat * 2); carve(&w->expanded, seen * exp * 2); carve(&w->zero_page, 4);
    carve(&w->proj, rows * round_up(proj, 32) * 4); carve(&w->mem, rows * mem * 4); carve(&w->y, 2 * rows * y_ld * 4);
    carve(&w->U, chunks * uf * 4); carve(&w->UN, chunks * nf * 4); carve(&w->gm, chunks * hm * 8); carve(&w->m_live, hm * 4); carve(&w->m_start, chunks * hm * 4);
    carve(&w->xn, 2 * rows * D * 2); carve(&w->attn, 2 * rows * kl * 2); carve(&w->memn, 2 * rows * kr * 2); carve(&w->q, 2 * rows * q * 2);
    carve(&w->gate, 2 * std::max(rows * gate, w->perm_rows * moe_ff) * 2);
    carve(&w->logits, rows * round_up(experts, 32) * 4); carve(&w->sel_w, rows * top * 4); carve(&w->sel_ids, rows * top * 4); carve(&w->slots, rows * top * 4);
    carve(&w->tile_group, std::max(w->max_tiles, 1) * 4); carve(&w->perm, 2 * w->perm_rows * D * 2); carve(&w->yp, w->perm_rows * y_ld * 4);
    cudaError_t e = cudaMalloc(&w->arena, off);
    if (e == cudaSuccess) e = cudaMemsetAsync(w->arena, 0, off, m->stream);
    if (e != cudaSuccess) return cuda_fail(e);
    for (auto& pr : places) *pr.first = (char*)w->arena + pr.second;
    w->rows = rows;
    w->seen = seen;
    return CD_OK;
}

// rows of one piece: x holds their embeddings, and their residual stream afterwards
template <typename KT>
int run_piece(cd_model* m, HybridPrefill* w, float* x, const uint32_t* ids, int rows, int pos0, bool split) {
    cd_hybrid_state& S = *m->hybrid;
    const int D = m->cfg.dim, y_ld = (int)round_up(D, 32), side = S.cfg.side_dim, nruns = (int)S.runs.size(), width = S.cfg.width;
    const float mult = S.cfg.residual_mult, eps = S.cfg.eps;
    typedef __nv_bfloat16 AT;
    const size_t R = w->rows;
    AT* xn = w->xn;
    AT* xn_lo = split ? xn + R * D : nullptr;
    Gemm gemm{m, w, split};
    auto check = [&](const char* what) {
        m->launches++;
        if (gemm.ok()) { gemm.e = cudaGetLastError(); gemm.what = what; }
    };
    // residual stream behind y and the operand of the linear that follows: `pre` of it
    auto settle = [&](const char* what, const float* y, const VecNorm& post, const VecNorm& pre, const float* add = nullptr, const int* slots = nullptr, int top = 0) {
        residual_rows_kernel<AT><<<rows, 256, D * 4, m->stream>>>(ResidualRows{x, y, y_ld, slots, w->sel_w, top, post, add, pre, mult, eps, width, D}, xn, xn_lo);
        check(what);
    };
    settle("embedding rows", nullptr, VecNorm{}, S.layers[S.runs[0].layer].pre1, S.step_vector(S.runs[0]));
    for (int r = 0; r < nruns && gemm.ok(); ++r) {
        const cd_hybrid_layer& L = S.layers[S.runs[r].layer];
        const FfnCfg& f = L.cfg.mlp;
        const bool pair = L.cfg.mixer == HybridLayerCfg::PARALLEL;
        // what the layer's last linear is followed by
        const VecNorm next_pre = r + 1 < nruns ? S.layers[S.runs[r + 1].layer].pre1 : VecNorm{};
        const float* next_add = r + 1 < nruns ? S.step_vector(S.runs[r + 1]) : nullptr;
        const VecNorm behind_ffn = side ? VecNorm{} : next_pre, behind_mixer = f.kind != FfnCfg::NONE ? L.pre2 : behind_ffn;
        const float *add_ffn = side ? nullptr : next_add, *add_mixer = f.kind != FfnCfg::NONE ? nullptr : add_ffn;
        const ProjLayout& pl = L.proj;
        const int proj_ld = (int)round_up(pl.rows, 32);
        const int activated = L.md.linear() ? pl.rg : 0;  // q, k and v of a linear attention
        gemm("projections", xn, xn_lo, L.wmix, rows, pl.rows, D, pl.rows, PfEpiPartial{w->proj, proj_ld, activated});
        KT* q = (KT*)w->q;
        KT* pool = (KT*)m->layers[r].kv;
        AT* attn = w->attn;
        AT* attn_lo = split ? attn + R * (size_t)L.kl : nullptr;
        AT* memn = w->memn;
        const int km = pair ? L.kr : L.kl;
        AT* memn_lo = split ? memn + R * (size_t)km : nullptr;
        // ---- attention
        if (L.cfg.has_attn()) {
            KT* q_lo = q + R * (size_t)L.ad.H * L.ad.kr();
            attn_rows_kernel<KT><<<rows, 256, 0, m->stream>>>(w->proj, proj_ld, L.ad, pl, L.q_norm, L.k_norm, m->page_table, pool, q, q_lo, pos0);
            check("query and key rows");
            const bool two = L.ad.maps == 2;
            const AttnWindow aw{L.ad, L.slopes, L.sink, w->proj, proj_ld, pl.lg, m->page_table, rows, pos0, L.kl, two ? w->raw : nullptr};
            if (gemm.ok()) { gemm.e = launch_attn_window<KT>(m, aw, q, q_lo, pool, attn, attn_lo); gemm.what = "attention"; }
            if (two) {
                diff_rows_kernel<AT><<<rows, 256, 0, m->stream>>>(w->raw, w->proj, proj_ld, pl.lg, L.ad, attn, attn_lo, L.kl);
                check("difference of the maps");
            }
        }
        // ---- latent attention: keys and values of all visible positions expanded first
        if (L.cfg.mixer == HybridLayerCfg::LATENT) {
            const MlaDims& d = L.ld;
            const AttnDims xd = expanded_dims(L, (int)w->seen);
            const int base = d.window > 0 ? std::max(0, pos0 - d.window + 1) : 0, n = pos0 + rows - base, cols = d.heads * (d.nope_n + d.vdim);
            KT* q_lo = q + R * (size_t)xd.H * xd.kp;
            KT* expanded = (KT*)w->expanded;
            AT* lat_lo = split ? w->latent + w->seen * (size_t)d.latent : nullptr;
            latent_rows_kernel<KT><<<rows, 256, 0, m->stream>>>(w->proj + pl.lq, proj_ld, d, Rotation{nullptr, L.freq, d.rot_dims}, L.latent_norm, m->page_table, pool, q, q_lo, xd.kp, pos0);
            check("query and latent rows");
            latent_gather_kernel<KT, AT><<<n, 256, 0, m->stream>>>(pool, m->page_table, d, base, w->latent, lat_lo, expanded, xd);
            check("cached latents");
            gemm("keys and values", w->latent, lat_lo, L.wukv, n, cols, d.latent, cols, PfEpiExpand<KT>{expanded, xd, d.nope_n});
            const AttnWindow aw{xd, nullptr, nullptr, nullptr, 0, 0, w->zero_page, rows, pos0 - base, L.kl, nullptr};
            if (gemm.ok()) { gemm.e = launch_attn_window<KT>(m, aw, q, q_lo, expanded, attn, attn_lo); gemm.what = "latent attention"; }
        }
        // ---- matrix memory, linear attention
        if (L.cfg.has_mem()) {
            MemPrompt mp;
            mp.d = L.md; mp.pl = pl; mp.proj = w->proj; mp.proj_ld = proj_ld; mp.ib = L.ib; mp.fb = L.fb; mp.rows = rows; mp.nchunk = (rows + MEM_CHUNK - 1) / MEM_CHUNK;
            mp.state = S.state + S.state_off[r]; mp.U = w->U; mp.UN = w->UN; mp.gm = w->gm; mp.m_live = w->m_live; mp.out = w->mem;
            const int vblocks = (L.md.vdim + 63) / 64, kblocks = (L.md.dim + 63) / 64;
            mem_chunk_kernel<<<dim3(mp.nchunk, L.md.H, vblocks * kblocks), 128, 0, m->stream>>>(mp, vblocks);
            check("memory contributions");
            mem_scan_kernel<<<dim3((unsigned)(((size_t)L.md.dim * L.md.vs / 4 + 255) / 256 + 1), L.md.H), 256, 0, m->stream>>>(mp, w->m_start);
            check("memory scan");
            if (gemm.ok()) gemm.e = cudaFuncSetAttribute(mem_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MEM_OUT_SMEM);
            mem_out_kernel<<<dim3(mp.nchunk, L.md.H, vblocks), 128, MEM_OUT_SMEM, m->stream>>>(mp, w->m_start);
            check("memory read-out");
            mem_rows_kernel<AT><<<rows, 256, 0, m->stream>>>(w->mem, w->proj, proj_ld, pl.rg, L.md, L.mem_norm, memn, memn_lo, km);
            check("memory rows");
        }
        // ---- output projections, norms, residual
        if (pair) {
            float *yl = w->y, *yr = w->y + R * (size_t)y_ld;
            gemm("attention output", attn, attn_lo, L.wo_l, rows, D, L.kl, D, PfEpiPartial{yl, y_ld});
            gemm("memory output", memn, memn_lo, L.wo_r, rows, D, L.kr, D, PfEpiPartial{yr, y_ld});
            parallel_mix_rows_kernel<AT><<<rows, 256, D * 4, m->stream>>>(x, yl, yr, y_ld, L.out_l, L.out_r, L.post1.w, mult, eps, width, D, xn, xn_lo);
            check("residual behind the mixers");
        } else {
            const bool mem = L.cfg.mixer == HybridLayerCfg::MEMORY;
            gemm("mixer output", mem ? memn : attn, mem ? memn_lo : attn_lo, L.wo_l, rows, D, L.kl, D, PfEpiPartial{w->y, y_ld});
            settle("residual behind the mixer", w->y, L.post1, behind_mixer, add_mixer);
        }
        // ---- feed-forward
        AT* gate = w->gate;
        if (f.kind == FfnCfg::DENSE) {
            AT* gate_lo = split ? gate + R * (size_t)L.ffp : nullptr;
            gemm("gate and up", xn, xn_lo, L.w13, rows, 2 * L.ffp, D, (size_t)2 * L.ffp, PfEpiGate<AT>{gate, gate_lo, L.ffp, CD_ACT_SWIGLU});
            gemm("down", gate, gate_lo, L.w2, rows, D, L.ffp, D, PfEpiPartial{w->y, y_ld});
            settle("residual behind the feed-forward", w->y, L.post2, behind_ffn, add_ffn);
        } else if (f.kind == FfnCfg::MOE) {
            const int z_ld = (int)round_up(f.experts, 32), n = rows * f.top;
            const int tiles = std::min(w->max_tiles, n / PF_BM + f.experts);
            gemm("router", xn, xn_lo, L.wr, rows, f.experts, D, f.experts, PfEpiPartial{w->logits, z_ld});
            const RouteRule rule{f.experts, f.top, f.groups, f.keep};
            route_rows_kernel<<<(rows + 3) / 4, 128, (size_t)4 * (f.experts + f.groups) * 4, m->stream>>>(w->logits, z_ld, rows, rule, w->sel_ids, w->sel_w);
            check("routing");
            plan_rows_kernel<<<1, 1024, f.experts * 4, m->stream>>>(w->sel_ids, n, f.experts, tiles, w->slots, w->tile_group);
            check("expert rows");
            AT* perm_lo = split ? w->perm + w->perm_rows * D : nullptr;
            gather_rows_kernel<AT><<<n, 128, 0, m->stream>>>(xn, xn_lo, w->slots, f.top, D, w->perm, perm_lo);
            check("expert row copies");
            AT* gate_lo = split ? gate + w->perm_rows * (size_t)L.ffp : nullptr;
            const int M = tiles * PF_BM;
            gemm("experts' gate and up", w->perm, perm_lo, L.w13, M, 2 * L.ffp, D, (size_t)f.experts * 2 * L.ffp, PfEpiGate<AT>{gate, gate_lo, L.ffp, CD_ACT_SWIGLU},
                 w->tile_group, 2 * L.ffp);
            gemm("experts' down", gate, gate_lo, L.w2, M, D, L.ffp, (size_t)f.experts * D, PfEpiPartial{w->yp, y_ld}, w->tile_group, D);
            settle("residual behind the experts", w->yp, L.post2, behind_ffn, add_ffn, w->slots, f.top);
        }
        // ---- token side
        if (side) {
            const int sp = S.side_pad();
            AT* side_lo = split ? w->side + R * (size_t)sp : nullptr;
            gemm("token side gate", xn, xn_lo, L.side_gate, rows, side, D, side,
                 PfEpiTokenGate<AT, AT>{w->side, side_lo, sp, (const AT*)S.side_embed + (size_t)S.runs[r].layer * side, S.side_ld(), side, ids});
            gemm("token side", w->side, side_lo, L.side_proj, rows, D, sp, D, PfEpiPartial{w->y, y_ld});
            settle("residual behind the token side", w->y, L.side_norm, next_pre, next_add);
        }
    }
    if (!gemm.ok()) return fail(m, CD_ERR_CUDA, std::string(gemm.what) + ": " + cudaGetErrorString(gemm.e));
    return CD_OK;
}

}  // namespace

int hybrid_prefill(cd_model* m, size_t n) {
    if (m->opt.weight_dtype != CD_DTYPE_BF16) return CD_ERR_UNSUPPORTED;
    cd_hybrid_state& S = *m->hybrid;
    if ((size_t)m->cfg.dim * 4 > 48 * 1024) return CD_ERR_UNSUPPORTED;  // a residual row is staged in shared memory
    for (const auto& L : S.layers) {
        const AttnDims a = L.cfg.mixer == HybridLayerCfg::LATENT ? expanded_dims(L, 1) : L.ad;
        if (a.vp > 256 || attn_window_smem(a.kp, a.vp) > 227 * 1024 || (L.cfg.mlp.kind == FfnCfg::MOE && (size_t)4 * (L.cfg.mlp.experts + L.cfg.mlp.groups) * 4 > 48 * 1024)) return CD_ERR_UNSUPPORTED;
    }
    HybridPrefill* w = (HybridPrefill*)S.prefill;
    if (!w) {
        S.prefill = w = new HybridPrefill();
        if (!(w->encode = encode_tiled_fn())) return fail(m, CD_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
    }
    size_t piece = PIECE_ROWS;
    if (const char* env = getenv("CD_PREFILL_ROWS")) piece = std::max<size_t>(1, strtoul(env, nullptr, 10));
    const char* mode = getenv("CD_PREFILL");
    const bool split = !(mode && !strcmp(mode, "fast"));
    int rc = ensure_workspace(m, w, n, piece);
    if (rc) return rc;
    m->state_len = SIZE_MAX;  // until the call has succeeded
    pf_embed_kernel<__nv_bfloat16><<<(unsigned)n, 256, 0, m->stream>>>((const __nv_bfloat16*)m->embed, m->prompt_dev, w->x, m->cfg.dim);
    m->launches++;
    for (size_t at = 0; at < n; at += piece) {
        float* x = w->x + at * m->cfg.dim;
        const int rows = (int)std::min(piece, n - at), pos0 = (int)(m->len + at);
        const uint32_t* ids = m->prompt_dev + at;
        rc = m->kv_dtype == CD_DTYPE_F16 ? run_piece<__half>(m, w, x, ids, rows, pos0, split) : run_piece<__nv_bfloat16>(m, w, x, ids, rows, pos0, split);
        if (rc) return rc;
    }
    const cudaError_t e = cudaMemcpyAsync(m->x_a, w->x + (n - 1) * (size_t)m->cfg.dim, (size_t)m->cfg.dim * 4, cudaMemcpyDeviceToDevice, m->stream);
    if (e != cudaSuccess) return fail(m, CD_ERR_CUDA, std::string("copy last row: ") + cudaGetErrorString(e));
    return CD_OK;
}

const float* hybrid_hidden_row(const cd_model* m, size_t i) { return static_cast<const HybridPrefill*>(m->hybrid->prefill)->x + i * (size_t)m->cfg.dim; }

void hybrid_prefill_release(cd_model* m) {
    HybridPrefill* w = (HybridPrefill*)m->hybrid->prefill;
    if (!w) return;
    if (w->x) cudaFree(w->x);
    if (w->arena) cudaFree(w->arena);
    delete w;
    m->hybrid->prefill = nullptr;
}

}  // namespace cd
