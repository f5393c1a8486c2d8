// A decoder whose layers a configuration file lists ("configured decoder"): per layer a mixer built from the mechanisms
// of mixers.cuh and a feed-forward, dense or a mixture of experts.  Host-side description, filled by the reader of one
// architecture (arch.cpp) and turned into device layers, cache rows and recurrent state by hybrid.cu.
#pragma once
#include <cuda_runtime.h>

#include <string>
#include <vector>

#include "mixers.cuh"
#include "model.h"
#include "moe.cuh"

namespace cd {

struct JsonValue;

// rotary positions on the first `dims` entries of a vector, in neighbouring pairs; angle = position * base^(-2 i / dims),
// under `scaled` with the long wavelengths stretched by `factor` (and a blend between original / high and original / low)
struct RotCfg {
    int dims = 0;
    double base = 10000.0;
    bool scaled = false;
    double factor = 1.0, low = 1.0, high = 1.0, original = 1.0;
};
std::vector<double> rot_frequencies(const RotCfg& r);

// softmax attention with the options the mechanisms of mixers.cuh know
struct AttnCfg {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    int window = 0;            // positions a query sees, itself included; 0: all
    float scale = 1.f;
    bool qk_norm = false;      // RMS norm of the whole q and k projections
    float temp_coef = 0.f;     // q *= 1 + coef * ln(floor((p + 1) / every) + 1); coef 0: off
    int temp_every = 1;
    bool distance_bias = false, sink = false;
    RotCfg rot;
    int maps = 1;              // 2: differential, two maps over the same values, the second one subtracted; per-head norm
    float diff = 0.f;
    enum Gate { GATE_NONE, GATE_HEAD, GATE_ELEMENT } gate = GATE_NONE;
};
// attention whose keys and values are linear in one normed latent per position, beside one rotated key part of all heads
struct LatentCfg {
    int heads = 0, dim = 0, rot_dim = 0, vdim = 0, rank = 0;
    int window = 0;
    float scale = 1.f;
    RotCfg rot;
};
// a [dim, vdim] state per head
struct MemCfg {
    enum Kind { MATRIX, LINEAR } kind = MATRIX;  // MATRIX: exponential input gate and forget gate (mLSTM); LINEAR: constant decay per head
    int heads = 0, dim = 0, vdim = 0;
    float gate_cap = 0.f;
    std::vector<double> decay;
};
struct FfnCfg {
    enum Kind { NONE, DENSE, MOE } kind = NONE;
    int ff = 0;                // columns of the dense FFN or of one expert
    int experts = 0, top = 0, groups = 1, keep = 1;
};
struct HybridLayerCfg {
    enum Mixer { PARALLEL, ATTENTION, MEMORY, LATENT } mixer = PARALLEL;  // PARALLEL: attn and mem side by side
    AttnCfg attn;
    MemCfg mem;
    LatentCfg latent;
    FfnCfg mlp;
    bool has_attn() const { return mixer == PARALLEL || mixer == ATTENTION; }
    bool has_mem() const { return mixer == PARALLEL || mixer == MEMORY; }
};
// one pass through a layer: each has its own cache rows and state
struct LayerRun {
    int layer;
    int step;                  // row of the loop's vectors added ahead of it, -1: none
};
struct HybridCfg {
    std::string architecture;
    int width = 0, vocab = 0;
    float eps = 1e-5f, residual_mult = 1.f;
    bool pre_norms = false;    // a norm ahead of each sublayer, beside the one behind it
    bool layer_norm = false;   // the model's norm: mean taken off, weight and bias; otherwise RMS with gain 1 + weight
    bool tied = false;         // the embedding table is the output matrix
    int side_dim = 0;          // columns per layer of the second embedding whose gated part every layer adds; 0: none
    int loop_start = 0, loop_stop = 0, loop_times = 0;  // layers start .. stop - 1 run `times` times in a row; times 0: no loop
    std::vector<HybridLayerCfg> layers;
    std::vector<LayerRun> runs() const;
};

// architecture name (config.json "architecture") -> reader of its configuration; false and *err on a bad one
struct ArchEntry {
    const char* name;
    bool (*parse)(const JsonValue& root, HybridCfg* out, std::string* err);
};
const ArchEntry* find_arch(const std::string& name);
bool parse_hybrid_config(const std::string& json_text, HybridCfg* out, std::string* err);

inline int pad_to(int v, int a) { return (v + a - 1) / a * a; }

}  // namespace cd

// one layer on the device
struct cd_hybrid_layer {
    cd::HybridLayerCfg cfg;
    cd::ProjLayout proj;         // where each projection sits in a row of `wmix`
    int kl = 0, kr = 0;          // columns of wo_l, wo_r (heads * vdim, padded to 8)
    int ffp = 0;                 // FFN columns padded to 16 (one expert's for a mixture)
    void *wmix = nullptr;        // [proj.rows][width]: every projection of the mixer's input, stacked
    void *wo_l = nullptr, *wo_r = nullptr;  // [width][kl], [width][kr]; a single mixer has the first only
    void *w13 = nullptr;         // dense: [2 ffp][width], rows (2j, 2j+1) = gate, up column j; experts: [experts][2 ffp][width]
    void *w2 = nullptr;          // [width][ffp]; experts: [experts][width][ffp]
    void *wr = nullptr;          // [experts][width]
    void *wuk_t = nullptr;       // latent attention: [heads][latent][nope], row (h, c) = column c of head h's key matrix
    void *wukv = nullptr;        // the same keys and the values as stored, [heads (dim + vdim)][latent]; fp32 models: the values only
    void *wuv = nullptr;         // its value rows
    void *side_gate = nullptr, *side_proj = nullptr;  // [side_dim][width], [width][side_dim padded to 8]
    // fp32 vectors
    float *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr, *slopes = nullptr;
    float *mem_norm = nullptr, *ib = nullptr, *fb = nullptr, *decay = nullptr, *log_decay = nullptr;
    float *out_l = nullptr, *out_r = nullptr;
    float *latent_norm = nullptr;
    double* freq = nullptr;      // angular frequencies of the rotation
    float lambda = 0.f;          // weight of the second attention map
    cd::VecNorm pre1{}, post1{}, pre2{}, post2{}, side_norm{};
    cd::AttnDims ad{};
    cd::MemDims md{};
    cd::MlaDims ld{};
    int nsplit = 1;              // attention slices of a decode step
    bool stream_ffn = true;      // the experts' rows go through the streamed GEMV (else: the plain-load kernels)
};

struct cd_hybrid_state {
    cd::HybridCfg cfg;
    std::vector<cd_hybrid_layer> layers;
    std::vector<cd::LayerRun> runs;
    std::vector<size_t> state_off;  // per run: its recurrent state inside a state slot (floats)
    cd::VecNorm final_norm{};
    float* loop_step = nullptr;     // [loop_times][width, padded]
    void* side_embed = nullptr;     // [vocab][layers * side_dim]
    const float* step_vector(const cd::LayerRun& r) const { return r.step < 0 ? nullptr : loop_step + (size_t)r.step * cd::pad_to(cfg.width, 8); }
    int side_ld() const { return (int)layers.size() * cfg.side_dim; }
    int side_pad() const { return cd::pad_to(cfg.side_dim, 8); }
    // recurrent state: slot 0 is the running sequence's, the others keep it at earlier lengths so that a session can
    // rewind (a cached row can be ignored, a state cannot be undone)
    float* state = nullptr;
    size_t slot_floats = 0;
    static constexpr int SLOTS = 5;
    static constexpr size_t FREE = (size_t)-1;
    size_t slot_len[SLOTS] = {FREE, FREE, FREE, FREE, FREE};  // [1..]: length the slot holds the state of
    uint64_t slot_used[SLOTS] = {0, 0, 0, 0, 0};
    uint64_t clock = 0;
    // scratch of a decode step
    void* ws = nullptr;
    float *proj = nullptr, *attn = nullptr, *mem = nullptr, *ssq = nullptr, *y = nullptr, *y2 = nullptr, *gate = nullptr, *side = nullptr, *zero = nullptr;
    float *part_acc = nullptr, *part_ml = nullptr, *router_logits = nullptr, *sel_w = nullptr, *loc_w = nullptr;
    float* qabs = nullptr;       // latent attention: absorbed queries, and the same as 16-bit heads and remainders
    void* qsplit = nullptr;
    unsigned int *counters = nullptr, *router_counter = nullptr;
    int *sel_ids = nullptr, *loc_ids = nullptr, *n_loc = nullptr;
    void* prefill = nullptr;     // workspace of the batched prompt pass (hybrid_prefill.cu)
};

namespace cd {
// batched prompt pass (hybrid_prefill.cu)
int hybrid_prefill(cd_model* m, size_t n);
const float* hybrid_hidden_row(const cd_model* m, size_t i);
void hybrid_prefill_release(cd_model* m);
}  // namespace cd
