// cd_model: device memory, the per-token launch sequence and the C ABI that mirrors
// metal_decode::Model (crates/metal-decode/src/lib.rs:129-511).
#include <algorithm>
#include <cmath>
#include <cstdio>
#include <cstring>

#include "step.cuh"

using namespace cd;

namespace {
thread_local std::string g_error;
}

namespace cd {
void set_global_error(const std::string& msg) { g_error = msg; }
int fail(cd_model* m, int code, const std::string& msg) {
    if (m) m->err = msg;
    g_error = msg;
    return code;
}
// A bounded device-side wait ran out (DevState::error holds where).  The word is cleared so the handle stays
// usable: the failed call's results are void, the cache length did not advance.
int device_wait_failed(cd_model* m, int dev_code, const char* where) {
    static const char* names[] = {"", "weight ring: stage never filled", "weight ring: stage never freed", "grid barrier", "tensor-parallel peer"};
    if (dev_code == DEV_ERR_BAD_TOKEN) {
        cudaMemsetAsync(&m->st->error, 0, sizeof(int32_t), m->stream);
        cudaStreamSynchronize(m->stream);
        return fail(m, CD_ERR_INVALID, std::string("the device selected a token id outside the vocabulary (logits without a finite maximum); row 0 was used") + where);
    }
    const char* what = dev_code >= 1 && dev_code <= 4 ? names[dev_code] : "tensor-core pipeline";
    cudaMemsetAsync(&m->st->error, 0, sizeof(int32_t), m->stream);
    cudaStreamSynchronize(m->stream);
    return fail(m, CD_ERR_DEVICE_WAIT, std::string("a bounded device-side wait ran out (") + what + ", code " + std::to_string(dev_code) + ")" + where);
}
}  // namespace cd

namespace {

__global__ void softcap_copy_kernel(const float* __restrict__ in, float* __restrict__ out, int n, float c) {
    const float inv = 1.0f / c;  // decode.rs:120-124: scale, tanh, scale
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) out[i] = c * tanhf(in[i] * inv);
}

cudaError_t enqueue_step(cd_model* m, const cd_step& p) { return m->family->enqueue_step(m, p); }

// Run one step: directly, or by replaying the captured graph of the same shape.
int run_step(cd_model* m, const cd_step& p) {
    m->state_len = SIZE_MAX;  // until the call has succeeded (advance)
    if (!m->opt.use_graph) {
        cudaError_t e = enqueue_step(m, p);
        if (e != cudaSuccess) return fail(m, CD_ERR_CUDA, std::string("step launch: ") + cudaGetErrorString(e));
        return CD_OK;
    }
    const cd_graph_key key{p.head, p.k, p.input, p.t, p.inv_t, p.softcap};
    auto it = m->graphs.find(key);
    if (it == m->graphs.end()) {
        const uint64_t before = m->launches;
        cudaGraph_t graph = nullptr;
        CK(m, cudaStreamBeginCapture(m->stream, cudaStreamCaptureModeThreadLocal));
        cudaError_t e = enqueue_step(m, p);
        cudaError_t e2 = cudaStreamEndCapture(m->stream, &graph);
        if (e != cudaSuccess || e2 != cudaSuccess) {
            if (graph) cudaGraphDestroy(graph);
            return fail(m, CD_ERR_CUDA, std::string("graph capture: ") + cudaGetErrorString(e != cudaSuccess ? e : e2));
        }
        cudaGraphExec_t exec = nullptr;
        CK(m, cudaGraphInstantiate(&exec, graph, 0));
        cudaGraphDestroy(graph);
        const cd_graph_entry entry{exec, m->launches - before};
        m->launches = before;
        it = m->graphs.emplace(key, entry).first;
    }
    CK(m, cudaGraphLaunch(it->second.exec, m->stream));
    m->launches += it->second.nodes;
    return CD_OK;
}

// the call succeeded: n more tokens are cached
void advance(cd_model* m, size_t n) {
    m->len += n;
    m->state_len = m->len;
}

}  // namespace

namespace cd {
// Counts a launch; in profiling mode also drops an event behind it so the time since
// the previous event can be charged to the launch's class.
void count_launch(cd_model* m) {
    m->launches++;
    if (m->profiling) {
        cudaEvent_t ev;
        cudaEventCreate(&ev);
        cudaEventRecord(ev, m->stream);
        m->prof_events.push_back(ev);
        m->prof_classes.push_back(m->cur_cls);
    }
}

int check_room(cd_model* m, size_t need) {
    if (m->tp_world > 1 && !m->tp_connected)
        return fail(m, CD_ERR_INVALID, "tensor-parallel model is not connected to its peers (cd_tp_connect)");
    if (m->len + need > (size_t)m->cfg.seq)
        return fail(m, CD_ERR_SEQ_FULL, "metal decode only supports lengths within cfg.seq");
    if (m->family->rewind && m->state_len != m->len)
        return fail(m, CD_ERR_INVALID, "the recurrent state is not the one at the cached length (an earlier call failed): cd_set_len to a length whose state is kept, or to 0");
    return CD_OK;
}
static int check_token(cd_model* m, uint32_t tok) {
    if (tok >= (uint32_t)m->cfg.vocab) return fail(m, CD_ERR_TOKEN, "token id must fit vocab for metal decode");
    return CD_OK;
}

int set_state(cd_model* m, uint32_t token) {
    // {pos, token} are the first 8 bytes of DevState: one small copy from pinned memory.
    // Every per-token entry point synchronises before returning, so the staging words are free.
    m->h_in[0] = (uint32_t)m->len;
    m->h_in[1] = token;
    CK(m, cudaMemcpyAsync(m->st, m->h_in, 8, cudaMemcpyHostToDevice, m->stream));
    return CD_OK;
}

}  // namespace cd

// ====================================================================== construction
namespace cd {

// the KV cache's storage: fp32 with fp32 weights, otherwise 16 bits (fp16 unless bf16 is asked for)
int resolve_kv_dtype(const cd_options& opts, int* kv_dtype) {
    const int wdt = opts.weight_dtype;
    int kvdt;
    switch (opts.kv_dtype) {
        case CD_KV_AUTO: kvdt = wdt == CD_DTYPE_F32 ? CD_DTYPE_F32 : CD_DTYPE_F16; break;
        case CD_KV_F32: kvdt = CD_DTYPE_F32; break;
        case CD_KV_F16: kvdt = CD_DTYPE_F16; break;
        case CD_KV_BF16: kvdt = CD_DTYPE_BF16; break;
        default: return fail(nullptr, CD_ERR_INVALID, "unknown KV-cache dtype");
    }
    if ((wdt == CD_DTYPE_F32) != (kvdt == CD_DTYPE_F32) || (wdt == CD_DTYPE_F16 && kvdt != CD_DTYPE_F16))
        return fail(nullptr, CD_ERR_UNSUPPORTED, "KV-cache dtype: fp32 goes with fp32 weights, fp16 with fp16 weights, fp16 or bf16 with bf16 / FP8 / INT4 weights");
    *kv_dtype = kvdt;
    return CD_OK;
}

int model_alloc(const cd_config* cfg, const cd_options& opts, int untied, const AllocSpec& spec, cd_model** out) {
    *out = nullptr;
    const int tpw = std::max(1, (int)opts.tp_world), tpr = tpw > 1 ? (int)opts.tp_rank : 0;
    int kvdt = 0;
    int rc = resolve_kv_dtype(opts, &kvdt);
    if (rc) return rc;
    cd_model* m = new cd_model();
    m->full_cfg = *cfg;
    m->cfg = spec.local;
    m->family = spec.family;
    m->replicated_head = !spec.sharded_head;
    m->tp_world = tpw;
    m->tp_rank = tpr;
    {
        // the LM head is split by vocabulary blocks under tensor parallelism and replicated under expert parallelism
        const int hw = spec.sharded_head ? tpw : 1, hr = spec.sharded_head ? tpr : 0;
        const int nblk = (cfg->vocab + HEAD_BLOCK - 1) / HEAD_BLOCK, per = (nblk + hw - 1) / hw;
        m->v0 = std::min(cfg->vocab, hr * per * HEAD_BLOCK);
        m->v_loc = std::min(cfg->vocab - m->v0, per * HEAD_BLOCK);
        m->tp_nb = per;  // head blocks per rank in the candidate exchange (the last rank may own fewer)
        if (m->v_loc <= 0) { delete m; return fail(nullptr, CD_ERR_UNSUPPORTED, "vocabulary too small for this tensor-parallel world size"); }
    }
    m->opt = opts;
    m->kv_dtype = kvdt;
    m->untied = untied;
    auto bail = [&](int code) { cd_model_destroy(m); return code; };
#define CKB(call) do { cudaError_t e_ = (call); if (e_ != cudaSuccess) { fail(nullptr, CD_ERR_CUDA, std::string(#call) + ": " + cudaGetErrorString(e_)); return bail(CD_ERR_CUDA); } } while (0)
    int ndev = 0;
    CKB(cudaGetDeviceCount(&ndev));
    if (ndev == 0) { fail(nullptr, CD_ERR_CUDA, "no CUDA device"); return bail(CD_ERR_CUDA); }
    if (opts.device >= 0) CKB(cudaSetDevice(opts.device));
    CKB(cudaGetDevice(&m->device));
    cudaDeviceProp prop;
    CKB(cudaGetDeviceProperties(&prop, m->device));
    m->sm_count = prop.multiProcessorCount;
    CKB(cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking));
    CKB(cudaEventCreate(&m->ev0));
    CKB(cudaEventCreate(&m->ev1));

    const cd_config& c = m->cfg;
    const size_t es = esize(is_quant(opts.weight_dtype) ? CD_DTYPE_BF16 : opts.weight_dtype), kes = esize(kvdt);
    m->alpha = 1.0f / std::sqrt(2.0f * (float)c.nlayers);  // lib.rs:201
    m->page_tokens = opts.page_tokens > 0 ? opts.page_tokens : 64;
    m->pages_per_seq = (c.seq + m->page_tokens - 1) / m->page_tokens;
    const int max_samples = std::max(1, opts.max_samples);
    m->num_pages = m->pages_per_seq * max_samples;
    m->nsplit = std::max(1, std::min(32, m->pages_per_seq));  // a slice is at most a few pages: one or two load rounds per CTA
    m->pdl = (opts.test_flags & 1) == 0;
    if (opts.test_ring_kb > 0) m->ring_kb = std::max(16, std::min(220, (int)opts.test_ring_kb));
    m->wait_ns = (unsigned long long)(opts.wait_us > 0 ? opts.wait_us : 2000000) * 1000ull;
    m->nblocks = (m->v_loc + HEAD_BLOCK - 1) / HEAD_BLOCK;  // head blocks of this rank's vocabulary shard

    // ---- embedding, LM head, final gamma
    const size_t D = c.dim, Q = c.q_dim, H = c.hidden, V = c.vocab;
    size_t off = 0;
    auto carve = [&](size_t bytes) { size_t o = off; off = align_up(off + bytes, 256); return o; };
    const size_t o_embed = carve(V * D * es);
    const size_t o_head = untied ? carve((size_t)m->v_loc * D * es) : o_embed + (size_t)m->v0 * D * es;  // tied: rows of the embedding
    const size_t o_gf = carve(D * 4);
    m->weight_bytes = off;
    CKB(cudaMalloc(&m->weight_arena, off));
    char* wb = (char*)m->weight_arena;
    m->embed = wb + o_embed; m->lm_head = wb + o_head; m->gamma_final = (float*)(wb + o_gf);
    m->layers.resize(c.nlayers);
    // ---- KV pages, a run per layer
    {
        size_t kv_bytes = 0;
        std::vector<size_t> at(c.nlayers);
        for (int l = 0; l < c.nlayers; ++l) {
            at[l] = kv_bytes;
            kv_bytes += align_up((size_t)m->num_pages * m->page_tokens * spec.kv_row_elems[l] * kes, 256);
        }
        CKB(cudaMalloc(&m->kv_arena, std::max<size_t>(kv_bytes, 256)));
        CKB(cudaMemsetAsync(m->kv_arena, 0, kv_bytes, m->stream));
        for (int l = 0; l < c.nlayers; ++l) m->layers[l].kv = (char*)m->kv_arena + at[l];
    }
    // ---- workspace
    off = 0;
    const size_t o_xa = carve(D * 4), o_xb = carve(D * 4), o_q = carve(Q * 4), o_attn = carve(Q * 4), o_gate = carve(H * 4);
    const size_t o_logits = carve(V * 4), o_logits2 = carve(V * 4), o_norm = carve(D * 4);
    const size_t nparts = std::max(m->nsplit, spec.attn_parts);  // attention partials per head: split-K slices, or what the family's own kernel needs
    const size_t o_pacc = carve((size_t)c.heads * nparts * c.hd * 4), o_pml = carve((size_t)c.heads * nparts * 2 * 4);
    const size_t o_cnt = carve((c.heads + 2) * 4);  // attention arrivals per head, head-kernel arrivals, pushing-GEMV arrivals
    const size_t o_bv = carve(m->nblocks * 4), o_bi = carve(m->nblocks * 4);
    const size_t o_tv = carve((size_t)m->nblocks * CD_MAX_GPU_TOPK * 4), o_ti = carve((size_t)m->nblocks * CD_MAX_GPU_TOPK * 4);
    const size_t o_mx = carve(m->nblocks * 4), o_sm = carve(m->nblocks * 4);
    const size_t o_tok = carve(256), o_ring = carve((c.seq + 1) * 4), o_prompt = carve((c.seq + 1) * 4);
    const size_t o_st = carve(sizeof(DevState)), o_pt = carve((size_t)m->num_pages * 4);
    const int rope_hd = spec.rope_dim;
    const size_t o_rope = carve((size_t)c.seq * (rope_hd / 2) * sizeof(float2));
    const size_t o_gc = carve(64), o_fam = carve(spec.family_ws_bytes);
    const size_t o_gv = carve((size_t)tpw * m->tp_nb * CD_MAX_GPU_TOPK * 4), o_gi = carve((size_t)tpw * m->tp_nb * CD_MAX_GPU_TOPK * 4);
    CKB(cudaMalloc(&m->ws_arena, off));
    CKB(cudaMemsetAsync(m->ws_arena, 0, off, m->stream));
    char* ws = (char*)m->ws_arena;
    m->x_a = (float*)(ws + o_xa); m->x_b = (float*)(ws + o_xb); m->q = (float*)(ws + o_q); m->attn = (float*)(ws + o_attn);
    m->gate = (float*)(ws + o_gate); m->logits = (float*)(ws + o_logits); m->logits_capped = (float*)(ws + o_logits2); m->norm_final = (float*)(ws + o_norm);
    m->part_acc = (float*)(ws + o_pacc); m->part_ml = (float*)(ws + o_pml); m->counters = (unsigned int*)(ws + o_cnt);
    m->block_vals = (float*)(ws + o_bv); m->block_idxs = (uint32_t*)(ws + o_bi);
    m->topk_vals = (float*)(ws + o_tv); m->topk_idxs = (uint32_t*)(ws + o_ti);
    m->maxes = (float*)(ws + o_mx); m->sums = (float*)(ws + o_sm);
    m->out_token = (uint32_t*)(ws + o_tok); m->out_ring = (uint32_t*)(ws + o_ring); m->prompt_dev = (uint32_t*)(ws + o_prompt);
    m->st = (DevState*)(ws + o_st); m->page_table = (int*)(ws + o_pt); m->rope = (float2*)(ws + o_rope);
    m->grid_counter = (unsigned long long*)(ws + o_gc); m->family_ws = ws + o_fam;
    m->tp_topk_vals = (float*)(ws + o_gv); m->tp_topk_idxs = (uint32_t*)(ws + o_gi);

    // identity page table; RoPE table from the host libm (sdpa_fwd.rs:18-33)
    {
        std::vector<int> pt(m->num_pages);
        for (int i = 0; i < m->num_pages; ++i) pt[i] = i;
        CKB(cudaMemcpyAsync(m->page_table, pt.data(), pt.size() * 4, cudaMemcpyHostToDevice, m->stream));
        std::vector<float2> rt((size_t)c.seq * (rope_hd / 2));
        for (int p = 0; p < c.seq; ++p)
            for (int i = 0; i < rope_hd / 2; ++i) {
                const float theta = (float)p / std::pow(10000.0f, 2.0f * (float)i / (float)rope_hd);
                rt[(size_t)p * (rope_hd / 2) + i] = make_float2(std::cos(theta), std::sin(theta));
            }
        if (rope_hd > 0) CKB(cudaMemcpyAsync(m->rope, rt.data(), rt.size() * sizeof(float2), cudaMemcpyHostToDevice, m->stream));
        CKB(cudaStreamSynchronize(m->stream));
    }
    CKB(cudaMallocHost(&m->h_ring, (c.seq + 1) * 4));
    CKB(cudaMallocHost(&m->h_state, sizeof(DevState)));
    CKB(cudaMallocHost(&m->h_in, 16));
    if (tpw > 1) {  // the region the peers write into: its own allocation, so it can be shared through CUDA IPC
        m->tp_pf_rows = spec.tp_prefill_rows;
        const size_t bytes = TpRegion::bytes_with_prefill(tpw, c.dim, m->tp_nb, m->tp_pf_rows);
        CKB(cudaMalloc((void**)&m->link_region, bytes));
        CKB(cudaMemset(m->link_region, 0, bytes));
        CKB(cudaMemset(m->link_region, 0xff, TpRegion::cand_off(tpw, c.dim)));  // inbox: every word "not arrived"
        m->tp.world = tpw; m->tp.rank = tpr; m->tp.dim = c.dim; m->tp.st = m->st; m->tp.wait_ns = m->wait_ns;
        m->tp.peers[tpr] = m->link_region;
    }
    {   // gammas default to 1 (LayerWeights::random, layer.rs:711-712)
        std::vector<float> ones(D, 1.0f);
        CKB(cudaMemcpy(m->gamma_final, ones.data(), D * 4, cudaMemcpyHostToDevice));
    }
#undef CKB
    *out = m;
    return CD_OK;
}
int model_finish(cd_model* m) {
    CK(m, cudaStreamSynchronize(m->stream));
    if (m->staging) { cudaFree(m->staging); m->staging = nullptr; m->staging_bytes = 0; }
    if (m->staging2) { cudaFree(m->staging2); m->staging2 = nullptr; m->staging2_bytes = 0; }
    return CD_OK;
}

}  // namespace cd

// ====================================================================== C ABI
extern "C" {

const char* cd_last_error(const cd_model* m) { return m ? m->err.c_str() : g_error.c_str(); }

void cd_model_destroy(cd_model* m) {
    if (!m) return;
    if (m->stream) cudaStreamSynchronize(m->stream);
    if (m->family && m->family->release) m->family->release(m);
    for (auto& kv : m->graphs) cudaGraphExecDestroy(kv.second.exec);
    for (int r = 0; r < 8; ++r) if (m->peer_maps[r]) cudaIpcCloseMemHandle(m->peer_maps[r]);
    if (m->link_region) cudaFree(m->link_region);
    if (m->weight_arena) cudaFree(m->weight_arena);
    if (m->layer_arena) cudaFree(m->layer_arena);
    if (m->kv_arena) cudaFree(m->kv_arena);
    if (m->ws_arena) cudaFree(m->ws_arena);
    if (m->staging) cudaFree(m->staging);
    if (m->staging2) cudaFree(m->staging2);
    if (m->h_ring) cudaFreeHost(m->h_ring);
    if (m->h_state) cudaFreeHost(m->h_state);
    if (m->h_in) cudaFreeHost(m->h_in);
    if (m->ev0) cudaEventDestroy(m->ev0);
    if (m->ev1) cudaEventDestroy(m->ev1);
    if (m->stream) cudaStreamDestroy(m->stream);
    delete m;
}

int cd_model_get_config(const cd_model* m, cd_config* cfg, cd_options* opts, int* untied) {
    if (!m) return CD_ERR_INVALID;
    if (cfg) *cfg = m->full_cfg;
    if (opts) *opts = m->opt;
    if (untied) *untied = m->untied;
    return CD_OK;
}

// ---- tensor parallel plumbing: one process per GPU, link regions exchanged through CUDA IPC
int cd_tp_region_handle(cd_model* m, void* out, size_t cap) {
    if (!m || !out) return fail(m, CD_ERR_INVALID, "null argument");
    if (m->tp_world <= 1) return fail(m, CD_ERR_INVALID, "model was not created tensor-parallel");
    if (cap < sizeof(cudaIpcMemHandle_t)) return fail(m, CD_ERR_CAPACITY, "handle buffer too small (64 bytes)");
    cudaIpcMemHandle_t h;
    CK(m, cudaIpcGetMemHandle(&h, m->link_region));
    memcpy(out, &h, sizeof h);
    return CD_OK;
}

int cd_tp_connect(cd_model* m, const void* handles, int world) {
    if (!m || !handles) return fail(m, CD_ERR_INVALID, "null argument");
    if (world != m->tp_world) return fail(m, CD_ERR_INVALID, "handle count does not match the tensor-parallel world size");
    CK(m, cudaSetDevice(m->device));
    for (int r = 0; r < world; ++r) {
        if (r == m->tp_rank) continue;
        cudaIpcMemHandle_t h;
        memcpy(&h, (const char*)handles + (size_t)r * sizeof h, sizeof h);
        void* p = nullptr;
        CK(m, cudaIpcOpenMemHandle(&p, h, cudaIpcMemLazyEnablePeerAccess));
        m->peer_maps[r] = p;
        m->tp.peers[r] = (char*)p;
    }
    m->tp_connected = true;
    return CD_OK;
}

int cd_tp_region_ptr(cd_model* m, void** out) {
    if (!m || !out) return fail(m, CD_ERR_INVALID, "null argument");
    if (m->tp_world <= 1) return fail(m, CD_ERR_INVALID, "model was not created tensor-parallel");
    *out = m->link_region;
    return CD_OK;
}

int cd_tp_connect_ptrs(cd_model* m, void* const* regions, int world) {
    if (!m || !regions) return fail(m, CD_ERR_INVALID, "null argument");
    if (world != m->tp_world) return fail(m, CD_ERR_INVALID, "region count does not match the tensor-parallel world size");
    for (int r = 0; r < world; ++r) {
        if (!regions[r]) return fail(m, CD_ERR_INVALID, "null link region");
        if (r != m->tp_rank) m->tp.peers[r] = (char*)regions[r];
    }
    m->tp_connected = true;
    return CD_OK;
}

static int tp_guard(cd_model* m, bool supported) {
    if (m->tp_world <= 1) return CD_OK;
    if (!m->tp_connected) return fail(m, CD_ERR_INVALID, "tensor-parallel model is not connected to its peers (cd_tp_connect)");
    if (!supported) return fail(m, CD_ERR_UNSUPPORTED, "not available on a tensor-parallel model: use the greedy entry points");
    return CD_OK;
}

int cd_len(const cd_model* m, size_t* len) {
    if (!m || !len) return CD_ERR_INVALID;
    *len = m->len;
    return CD_OK;
}

int cd_set_len(cd_model* m, size_t len) {
    if (!m) return CD_ERR_INVALID;
    len = std::min(len, (size_t)m->cfg.seq);
    if (m->family->rewind) {  // cached rows can be ignored, a recurrent state has to be the one at that length
        const int rc = m->family->rewind(m, len);
        if (rc) return rc;
    }
    m->len = len;
    return CD_OK;
}

int cd_can_rewind(const cd_model* m, size_t len) {
    if (!m) return 0;
    return !m->family->can_rewind || m->family->can_rewind(m, len) ? 1 : 0;
}

// calls that start from a hidden state instead of a token id
static int hidden_input_guard(cd_model* m) {
    return m->needs_token ? fail(m, CD_ERR_UNSUPPORTED, "this model's layers read the token id: use the calls that take one") : (int)CD_OK;
}

int cd_decode_token(cd_model* m, const float* x_in, float* x_out) {
    if (m) { int g_ = tp_guard(m, false); if (g_) return g_; }
    if (!m || !x_in || !x_out) return fail(m, CD_ERR_INVALID, "null argument");
    if (int g_ = hidden_input_guard(m)) return g_;
    int rc = check_room(m, 1);
    if (rc) return rc;
    CK(m, cudaMemcpyAsync(m->x_a, x_in, (size_t)m->full_cfg.dim * 4, cudaMemcpyHostToDevice, m->stream));
    if ((rc = set_state(m, 0))) return rc;
    cd_step p{0, HEAD_NONE};
    if ((rc = run_step(m, p))) return rc;
    CK(m, cudaMemcpyAsync(x_out, m->x_a, (size_t)m->full_cfg.dim * 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaMemcpyAsync(&m->h_in[2], &m->st->error, 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaStreamSynchronize(m->stream));
    if (m->h_in[2]) return device_wait_failed(m, (int)m->h_in[2], "");
    advance(m, 1);
    return CD_OK;
}

int cd_decode_token_from_id(cd_model* m, uint32_t token, float* x_out) {
    if (m) { int g_ = tp_guard(m, false); if (g_) return g_; }
    if (!m || !x_out) return fail(m, CD_ERR_INVALID, "null argument");
    int rc = check_room(m, 1);
    if (rc) return rc;
    if ((rc = check_token(m, token))) return rc;
    if ((rc = set_state(m, token))) return rc;
    cd_step p{1, HEAD_NONE};
    if ((rc = run_step(m, p))) return rc;
    CK(m, cudaMemcpyAsync(x_out, m->x_a, (size_t)m->full_cfg.dim * 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaMemcpyAsync(&m->h_in[2], &m->st->error, 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaStreamSynchronize(m->stream));
    if (m->h_in[2]) return device_wait_failed(m, (int)m->h_in[2], "");
    advance(m, 1);
    return CD_OK;
}

static int argmax_common(cd_model* m, int input, uint32_t token, uint32_t* out) {
    int rc = set_state(m, token);
    if (rc) return rc;
    cd_step p{input, HEAD_ARGMAX};
    if ((rc = run_step(m, p))) return rc;
    CK(m, cudaMemcpyAsync(m->h_ring, m->out_token, 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaMemcpyAsync(&m->h_in[2], &m->st->error, 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaStreamSynchronize(m->stream));
    if (m->h_in[2]) return device_wait_failed(m, (int)m->h_in[2], "");
    *out = m->h_ring[0];
    advance(m, 1);
    return CD_OK;
}

int cd_decode_token_argmax(cd_model* m, const float* x_in, uint32_t* out) {
    if (!m || !x_in || !out) return fail(m, CD_ERR_INVALID, "null argument");
    if (int g_ = hidden_input_guard(m)) return g_;
    int rc = check_room(m, 1);
    if (rc) return rc;
    CK(m, cudaMemcpyAsync(m->x_a, x_in, (size_t)m->full_cfg.dim * 4, cudaMemcpyHostToDevice, m->stream));
    return argmax_common(m, 0, 0, out);
}

int cd_decode_token_argmax_from_id(cd_model* m, uint32_t token, uint32_t* out) {
    if (!m || !out) return fail(m, CD_ERR_INVALID, "null argument");
    int rc = check_room(m, 1);
    if (rc) return rc;
    if ((rc = check_token(m, token))) return rc;
    return argmax_common(m, 1, token, out);
}

int cd_decode_token_topk_from_id(cd_model* m, uint32_t token, size_t top_k, float* out_vals, uint32_t* out_idxs, size_t cap,
                                 size_t* count) {
    if (m) { int g_ = tp_guard(m, true); if (g_) return g_; }  // tensor parallel: every rank returns all ranks' candidates
    if (!m || !out_vals || !out_idxs || !count) return fail(m, CD_ERR_INVALID, "null argument");
    int rc = check_room(m, 1);
    if (rc) return rc;
    if ((rc = check_token(m, token))) return rc;
    if (top_k == 0) return fail(m, CD_ERR_INVALID, "top_k must be positive");
    if (top_k > CD_MAX_GPU_TOPK) return fail(m, CD_ERR_INVALID, "top_k exceeds metal decode top-k capacity");
    const int nblk_all = (m->full_cfg.vocab + HEAD_BLOCK - 1) / HEAD_BLOCK;  // == m->nblocks on one GPU
    const size_t n = (size_t)nblk_all * top_k;
    if (cap < n) return fail(m, CD_ERR_CAPACITY, "out_vals too small for top-k candidates");
    if ((rc = set_state(m, token))) return rc;
    cd_step p{1, HEAD_TOPK};
    p.k = (int)top_k;
    if ((rc = run_step(m, p))) return rc;
    if (m->tp_world > 1) {
        for (int r = 0; r < m->tp_world; ++r) {  // rank r's row of the gathered candidates holds its blocks, k entries each
            const int nb_r = std::min(m->tp_nb, nblk_all - r * m->tp_nb);
            if (nb_r <= 0) break;
            const size_t src = (size_t)r * m->tp_nb * 32, dst = (size_t)r * m->tp_nb * top_k, cnt = (size_t)nb_r * top_k * 4;
            CK(m, cudaMemcpyAsync(out_vals + dst, m->tp_topk_vals + src, cnt, cudaMemcpyDeviceToHost, m->stream));
            CK(m, cudaMemcpyAsync(out_idxs + dst, m->tp_topk_idxs + src, cnt, cudaMemcpyDeviceToHost, m->stream));
        }
    } else {
        CK(m, cudaMemcpyAsync(out_vals, m->topk_vals, n * 4, cudaMemcpyDeviceToHost, m->stream));
        CK(m, cudaMemcpyAsync(out_idxs, m->topk_idxs, n * 4, cudaMemcpyDeviceToHost, m->stream));
    }
    CK(m, cudaMemcpyAsync(&m->h_in[2], &m->st->error, 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaStreamSynchronize(m->stream));
    if (m->h_in[2]) return device_wait_failed(m, (int)m->h_in[2], "");
    *count = n;
    advance(m, 1);
    return CD_OK;
}

int cd_decode_token_block_stats_from_id(cd_model* m, uint32_t token, float inv_temperature, float softcap, float* out_maxes,
                                        float* out_sums, size_t cap, size_t* nblocks) {
    if (m) { int g_ = tp_guard(m, false); if (g_) return g_; }
    if (!m || !out_maxes || !out_sums || !nblocks) return fail(m, CD_ERR_INVALID, "null argument");
    int rc = check_room(m, 1);
    if (rc) return rc;
    if ((rc = check_token(m, token))) return rc;
    if (cap < (size_t)m->nblocks) return fail(m, CD_ERR_CAPACITY, "out_maxes too small");
    if ((rc = set_state(m, token))) return rc;
    cd_step p{1, HEAD_STATS};
    p.inv_t = inv_temperature;
    p.softcap = softcap;
    if ((rc = run_step(m, p))) return rc;
    CK(m, cudaMemcpyAsync(out_maxes, m->maxes, (size_t)m->nblocks * 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaMemcpyAsync(out_sums, m->sums, (size_t)m->nblocks * 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaMemcpyAsync(&m->h_in[2], &m->st->error, 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaStreamSynchronize(m->stream));
    if (m->h_in[2]) return device_wait_failed(m, (int)m->h_in[2], "");
    *nblocks = (size_t)m->nblocks;
    advance(m, 1);
    return CD_OK;
}

int cd_materialize_current_logits_block(cd_model* m, size_t block_idx, float softcap, float* out, size_t cap, size_t* valid) {
    if (m) { int g_ = tp_guard(m, false); if (g_) return g_; }
    if (!m || !out || !valid) return fail(m, CD_ERR_INVALID, "null argument");
    if (block_idx >= (size_t)m->nblocks) return fail(m, CD_ERR_INVALID, "block_idx out of range");
    const size_t n = std::min<size_t>(HEAD_BLOCK, (size_t)m->cfg.vocab - block_idx * HEAD_BLOCK);
    if (cap < n) return fail(m, CD_ERR_CAPACITY, "out_logits too small");
    // The logits of the last step are still resident (the reference recomputes them from the
    // resident normalised hidden, lib.rs:997); softcap without temperature as lib.rs:1716-1719.
    const float* src = m->logits + block_idx * HEAD_BLOCK;
    if (softcap > 0.0f) {
        float* tmp = m->logits_capped;
        softcap_copy_kernel<<<1, 256, 0, m->stream>>>(src, tmp, (int)n, softcap);
        count_launch(m);
        CK(m, cudaGetLastError());
        src = tmp;
    }
    CK(m, cudaMemcpyAsync(out, src, n * 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaStreamSynchronize(m->stream));
    *valid = n;
    return CD_OK;
}

static int fetch_logits(cd_model* m, float softcap, float* out) {
    const int V = m->cfg.vocab;
    const float* src = m->logits;
    if (softcap > 0.0f) {
        float* capped = m->logits_capped;
        softcap_copy_kernel<<<m->sm_count, 256, 0, m->stream>>>(m->logits, capped, V, softcap);
        count_launch(m);
        CK(m, cudaGetLastError());
        src = capped;
    }
    CK(m, cudaMemcpyAsync(out, src, (size_t)V * 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaStreamSynchronize(m->stream));
    return CD_OK;
}

int cd_decode_token_logits_from_id(cd_model* m, uint32_t token, float softcap, float* out_logits) {
    if (m) { int g_ = tp_guard(m, false); if (g_) return g_; }
    if (!m || !out_logits) return fail(m, CD_ERR_INVALID, "null argument");
    int rc = check_room(m, 1);
    if (rc) return rc;
    if ((rc = check_token(m, token))) return rc;
    if ((rc = set_state(m, token))) return rc;
    cd_step p{1, HEAD_LOGITS};
    if ((rc = run_step(m, p))) return rc;
    if ((rc = fetch_logits(m, softcap, out_logits))) return rc;
    advance(m, 1);
    return CD_OK;
}

// n prompt tokens behind the cached ones; row k of `out` receives the logits at place want[k] of them
static int prefill_impl(cd_model* m, const uint32_t* ids, size_t n, const size_t* want, size_t nwant, float softcap, float* out) {
    int rc = check_room(m, n);
    if (rc) return rc;
    for (size_t i = 0; i < n; ++i)
        if ((rc = check_token(m, ids[i]))) return rc;
    for (size_t k = 0; k < nwant; ++k)
        if (want[k] >= n) return fail(m, CD_ERR_INVALID, "a wanted place lies behind the last token");
    const size_t V = m->cfg.vocab;
    CK(m, cudaMemcpyAsync(m->prompt_dev, ids, n * 4, cudaMemcpyHostToDevice, m->stream));
    auto finish = [&](const char* where) {
        CK(m, cudaMemcpyAsync(m->h_state, m->st, sizeof(DevState), cudaMemcpyDeviceToHost, m->stream));
        CK(m, cudaStreamSynchronize(m->stream));
        CK(m, cudaEventElapsedTime(&m->last_ms, m->ev0, m->ev1));
        if (m->h_state->error) return device_wait_failed(m, m->h_state->error, where);
        advance(m, n);
        return m->family->mark ? m->family->mark(m) : (int)CD_OK;
    };
    // Prompts of a few tokens and up go through the batched tensor-core pass where the model
    // allows it (CD_PREFILL=token keeps the one-token-at-a-time path of inference.rs:650-670).
    const char* mode = getenv("CD_PREFILL");
    if (n >= 8 && m->family->prefill && !(mode && !strcmp(mode, "token"))) {
        CK(m, cudaEventRecord(m->ev0, m->stream));
        rc = m->family->prefill(m, n);
        if (rc == CD_OK) {
            begin_loop_kernel<<<1, 1, 0, m->stream>>>(m->st, (int)(m->len + n), 0u, 0ull);
            count_launch(m);
            for (size_t k = 0; k < nwant; ++k) {
                if (!(nwant == 1 && want[0] + 1 == n))  // the last row is in place
                    CK(m, cudaMemcpyAsync(m->x_a, m->family->hidden_row(m, want[k]), (size_t)m->cfg.dim * 4, cudaMemcpyDeviceToDevice, m->stream));
                cudaError_t e = m->family->enqueue_head_only(m);
                if (e != cudaSuccess) return fail(m, CD_ERR_CUDA, std::string("head launch: ") + cudaGetErrorString(e));
                if (k + 1 == nwant) CK(m, cudaEventRecord(m->ev1, m->stream));
                if ((rc = fetch_logits(m, softcap, out + k * V))) return rc;
            }
            if (nwant == 0) CK(m, cudaEventRecord(m->ev1, m->stream));
            return finish(" during the batched prompt pass");
        }
        if (rc != CD_ERR_UNSUPPORTED) return rc;
    }
    begin_loop_kernel<<<1, 1, 0, m->stream>>>(m->st, (int)m->len, 0u, 0ull);
    count_launch(m);
    CK(m, cudaEventRecord(m->ev0, m->stream));
    for (size_t i = 0; i < n; ++i) {
        const size_t* w = std::find(want, want + nwant, i);
        cd_step p{2, w != want + nwant ? HEAD_LOGITS : HEAD_NONE};
        if ((rc = run_step(m, p))) return rc;
        if (i + 1 == n) CK(m, cudaEventRecord(m->ev1, m->stream));
        for (; w != want + nwant; w = std::find(w + 1, want + nwant, i))
            if ((rc = fetch_logits(m, softcap, out + (size_t)(w - want) * V))) return rc;
    }
    return finish("");
}

int cd_prefill(cd_model* m, const uint32_t* ids, size_t n, float softcap, float* last_logits) {
    if (m) { int g_ = tp_guard(m, last_logits == nullptr); if (g_) return g_; }
    if (!m || !ids || n == 0) return fail(m, CD_ERR_INVALID, "prompt must contain at least one token");
    const size_t last = n - 1;
    return prefill_impl(m, ids, n, &last, last_logits ? 1 : 0, softcap, last_logits);
}

int cd_prefill_logits(cd_model* m, const uint32_t* ids, size_t n, const size_t* want, size_t nwant, float softcap, float* out) {
    if (m) { int g_ = tp_guard(m, nwant == 0); if (g_) return g_; }
    if (!m || !ids || n == 0) return fail(m, CD_ERR_INVALID, "prompt must contain at least one token");
    if (nwant && (!want || !out)) return fail(m, CD_ERR_INVALID, "null argument");
    return prefill_impl(m, ids, n, want, nwant, softcap, out);
}

static int decode_loop(cd_model* m, uint32_t first, size_t nsteps, cd_step p, uint64_t* rng, uint32_t* out_ids) {
    if (!m || !out_ids) return fail(m, CD_ERR_INVALID, "null argument");
    int rc = check_room(m, nsteps);
    if (rc) return rc;
    if ((rc = check_token(m, first))) return rc;
    if (nsteps == 0) return CD_OK;
    begin_loop_kernel<<<1, 1, 0, m->stream>>>(m->st, (int)m->len, first, rng ? *rng : 0ull);
    count_launch(m);
    CK(m, cudaGetLastError());
    CK(m, cudaEventRecord(m->ev0, m->stream));
    for (size_t i = 0; i < nsteps; ++i)
        if ((rc = run_step(m, p))) return rc;
    CK(m, cudaEventRecord(m->ev1, m->stream));
    CK(m, cudaMemcpyAsync(m->h_ring, m->out_ring, nsteps * 4, cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaMemcpyAsync(m->h_state, m->st, sizeof(DevState), cudaMemcpyDeviceToHost, m->stream));
    CK(m, cudaStreamSynchronize(m->stream));
    CK(m, cudaEventElapsedTime(&m->last_ms, m->ev0, m->ev1));
    if (m->h_state->error) return device_wait_failed(m, m->h_state->error, "");
    memcpy(out_ids, m->h_ring, nsteps * 4);
    if (rng) *rng = m->h_state->rng;
    advance(m, nsteps);
    return CD_OK;
}

int cd_decode_steps_greedy(cd_model* m, uint32_t first, size_t nsteps, uint32_t* out_ids) {
    cd_step p{1, LOOP_GREEDY};
    return decode_loop(m, first, nsteps, p, nullptr, out_ids);
}

int cd_decode_steps_topk(cd_model* m, uint32_t first, size_t nsteps, size_t top_k, float t, float softcap, uint64_t* rng,
                         uint32_t* out_ids) {
    if (m) { int g_ = tp_guard(m, true); if (g_) return g_; }  // tensor parallel: candidates are exchanged between the ranks
    if (!m || !rng) return fail(m, CD_ERR_INVALID, "null argument");
    if (top_k == 0 || top_k > CD_MAX_GPU_TOPK) return fail(m, CD_ERR_INVALID, "top_k exceeds metal decode top-k capacity");
    cd_step p{1, LOOP_TOPK};
    p.k = (int)std::min<size_t>(top_k, (size_t)m->cfg.vocab);  // decode.rs:140
    p.t = t;
    p.softcap = softcap;
    return decode_loop(m, first, nsteps, p, rng, out_ids);
}

int cd_decode_steps_fullvocab(cd_model* m, uint32_t first, size_t nsteps, float t, float softcap, uint64_t* rng,
                              uint32_t* out_ids) {
    if (m) { int g_ = tp_guard(m, true); if (g_) return g_; }  // tensor parallel: block statistics are exchanged between the ranks
    if (!m || !rng) return fail(m, CD_ERR_INVALID, "null argument");
    // (a vocabulary-sharded head exchanges one (max, sum) per block of every rank; the MoE model's head is replicated)
    if (m->nblocks > 256 || (!m->replicated_head && m->tp_world * m->tp_nb > 256)) return fail(m, CD_ERR_UNSUPPORTED, "full-vocab block sampler supports at most 65536 vocabulary rows");
    cd_step p{1, LOOP_FULLVOCAB};
    p.t = t;
    p.inv_t = 1.0f / std::max(t, 1.17549435e-38f);  // decode.rs:174
    p.softcap = softcap;
    return decode_loop(m, first, nsteps, p, rng, out_ids);
}

int cd_decode_steps_samples(cd_model* m, const uint32_t* first_tokens, size_t nsamples, size_t nsteps, int mode, size_t top_k,
                            float temperature, float softcap, uint64_t* rng_states, uint32_t* out_ids) {
    if (m) { int g_ = tp_guard(m, false); if (g_) return g_; }
    if (!m || !first_tokens || !out_ids) return fail(m, CD_ERR_INVALID, "null argument");
    if (nsamples == 0 || nsamples > 16 || nsamples > (size_t)(m->num_pages / m->pages_per_seq))
        return fail(m, CD_ERR_CAPACITY, "sample count exceeds cd_options.max_samples (at most 16)");
    if (mode < CD_SAMPLES_GREEDY || mode > CD_SAMPLES_FULLVOCAB) return fail(m, CD_ERR_INVALID, "unknown sampling mode");
    if (mode != CD_SAMPLES_GREEDY && !rng_states) return fail(m, CD_ERR_INVALID, "null argument");
    if (mode == CD_SAMPLES_TOPK && (top_k == 0 || top_k > CD_MAX_GPU_TOPK)) return fail(m, CD_ERR_INVALID, "top_k exceeds metal decode top-k capacity");
    if (mode == CD_SAMPLES_FULLVOCAB && m->nblocks > 256) return fail(m, CD_ERR_UNSUPPORTED, "full-vocab block sampler supports at most 65536 vocabulary rows");
    int rc = check_room(m, nsteps);
    if (rc) return rc;
    for (size_t s = 0; s < nsamples; ++s)
        if ((rc = check_token(m, first_tokens[s]))) return rc;
    if (nsteps == 0) return CD_OK;
    rc = !m->family->samples ? CD_ERR_UNSUPPORTED : m->family->samples(m, first_tokens, (int)nsamples, nsteps, mode, (int)std::min<size_t>(top_k, (size_t)m->cfg.vocab), temperature, softcap,
                        rng_states, out_ids);
    if (rc == CD_ERR_UNSUPPORTED) return fail(m, rc, "multi-sample decode needs a bf16 / fp16 single-GPU model");
    return rc;
}

int cd_profile_decode_step(cd_model* m, uint32_t token, float* ms_by_class, uint32_t* launches_by_class, size_t nclasses) {
    if (!m || !ms_by_class || !launches_by_class || nclasses < CLS_COUNT) return fail(m, CD_ERR_INVALID, "need room for 8 classes");
    int rc = check_room(m, 1);
    if (rc) return rc;
    if ((rc = check_token(m, token))) return rc;
    if ((rc = set_state(m, token))) return rc;
    CK(m, cudaStreamSynchronize(m->stream));
    m->profiling = true;
    m->prof_events.clear();
    m->prof_classes.clear();
    m->cur_cls = CLS_MISC;
    cudaEvent_t start;
    cudaEventCreate(&start);
    cudaEventRecord(start, m->stream);
    cd_step p{1, HEAD_ARGMAX};
    cudaError_t e = enqueue_step(m, p);
    m->profiling = false;
    cudaError_t e2 = cudaStreamSynchronize(m->stream);
    for (size_t i = 0; i < nclasses; ++i) { ms_by_class[i] = 0.f; launches_by_class[i] = 0; }
    cudaEvent_t prev = start;
    for (size_t i = 0; i < m->prof_events.size(); ++i) {
        float ms = 0.f;
        if (e == cudaSuccess && e2 == cudaSuccess) cudaEventElapsedTime(&ms, prev, m->prof_events[i]);
        ms_by_class[m->prof_classes[i]] += ms;
        launches_by_class[m->prof_classes[i]] += 1;
        if (prev != start) cudaEventDestroy(prev);
        prev = m->prof_events[i];
    }
    if (prev != start) cudaEventDestroy(prev);
    cudaEventDestroy(start);
    m->prof_events.clear();
    m->prof_classes.clear();
    if (e != cudaSuccess || e2 != cudaSuccess)
        return fail(m, CD_ERR_CUDA, std::string("profiled step: ") + cudaGetErrorString(e != cudaSuccess ? e : e2));
    advance(m, 1);
    return CD_OK;
}

int cd_debug_phase_trace(cd_model* m, unsigned long long* out, size_t cap, size_t* n) {
    if (!m || !out || !n) return CD_ERR_INVALID;
    const size_t count = (size_t)2 * (10 * m->cfg.nlayers + 2);
    if (!m->mega_trace) return fail(m, CD_ERR_UNSUPPORTED, "phase tracing is off (cd_options.test_flags bit 2 when the model is created)");
    if (cap < count) return fail(m, CD_ERR_CAPACITY, "trace buffer too small");
    CK(m, cudaMemcpy(out, m->mega_trace, count * 8, cudaMemcpyDeviceToHost));
    *n = count;
    return CD_OK;
}

int cd_last_device_ms(const cd_model* m, float* ms) {
    if (!m || !ms) return CD_ERR_INVALID;
    *ms = m->last_ms;
    return CD_OK;
}

int cd_kernel_launches(const cd_model* m, uint64_t* n) {
    if (!m || !n) return CD_ERR_INVALID;
    *n = m->launches;
    return CD_OK;
}

}  // extern "C"
