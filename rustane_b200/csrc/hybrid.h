// A decoder whose layers a configuration file lists ("configured decoder"): per layer a mixer built from the mechanisms
// of mixers.cuh and a feed-forward, dense or a mixture of experts.  Host-side description, filled by the reader of one
// architecture (arch.cpp) and turned into device layers, cache rows and recurrent state by hybrid.cu.
#pragma once
#include <cuda_runtime.h>

#include <string>
#include <vector>

#include "mixers.cuh"
#include "model.h"

namespace cd {

struct JsonValue;

// softmax attention with the options the mechanisms of mixers.cuh know
struct AttnCfg {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    int window = 0;            // positions a query sees, itself included; 0: all
    float scale = 1.f;
    float temp_coef = 0.f;     // q *= 1 + coef * ln(floor((p + 1) / every) + 1); coef 0: off
    int temp_every = 1;
};
// matrix memory with exponential input gate (mLSTM)
struct MemCfg {
    int heads = 0, dim = 0, vdim = 0;
    float gate_cap = 0.f;
};
struct FfnCfg {
    enum Kind { NONE, DENSE, MOE } kind = NONE;
    int ff = 0;                // columns of the dense FFN or of one expert
    int experts = 0, top = 0, groups = 1, keep = 1;
};
struct HybridLayerCfg {
    AttnCfg left;
    MemCfg right;
    FfnCfg mlp;
};
struct HybridCfg {
    std::string architecture;
    int width = 0, vocab = 0;
    float eps = 1e-5f, residual_mult = 1.f;
    std::vector<HybridLayerCfg> layers;
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
    void *wo_l = nullptr, *wo_r = nullptr;  // [width][kl], [width][kr]
    void *w13 = nullptr;         // dense: [2 ffp][width], rows (2j, 2j+1) = gate, up column j; experts: [experts][2 ffp][width]
    void *w2 = nullptr;          // [width][ffp]; experts: [experts][width][ffp]
    void *wr = nullptr;          // [experts][width]
    // fp32 vectors
    float *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr, *slopes = nullptr;
    float *mem_norm = nullptr, *ib = nullptr, *fb = nullptr;
    float *out_l = nullptr, *out_r = nullptr;
    float *gain1 = nullptr, *gain2 = nullptr;  // 1 + weight
    size_t state_off = 0;        // this layer's recurrent state inside a state slot (floats)
    cd::AttnDims ad;
    cd::MemDims md;
    int nsplit = 1;              // attention slices of a decode step
    bool stream_ffn = true;      // the experts' rows go through the streamed GEMV (else: the plain-load kernels)
};

struct cd_hybrid_state {
    cd::HybridCfg cfg;
    std::vector<cd_hybrid_layer> layers;
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
    float *proj = nullptr, *attn = nullptr, *mem = nullptr, *ssq = nullptr, *y = nullptr, *y2 = nullptr, *gate = nullptr, *zero = nullptr;
    float *part_acc = nullptr, *part_ml = nullptr, *router_logits = nullptr, *sel_w = nullptr, *loc_w = nullptr;
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
