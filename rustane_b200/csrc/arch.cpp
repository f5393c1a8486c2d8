// Registry of configured architectures: config.json's "architecture" names the reader that turns it into the layer
// description of hybrid.h.  Another design adds a reader here and, where it has one, a mechanism in mixers.cuh.
#include <cmath>
#include <cstring>

#include "hybrid.h"
#include "json.h"

namespace cd {
namespace {

// Reads fields of one object; the first failure is kept with the path of the field.
struct Fields {
    const JsonValue& v;
    std::string path;
    std::string* err;
    bool ok = true;
    void bad(const std::string& what) {
        if (ok && err->empty()) *err = path + ": " + what;
        ok = false;
    }
    const JsonValue* child(const char* key, bool required) {
        const JsonValue* c = v.get(key);
        if (!c && required) bad(std::string("missing \"") + key + "\"");
        if (c && c->kind != JsonValue::OBJ) { bad(std::string("\"") + key + "\" must be an object"); return nullptr; }
        return c;
    }
    void number(const char* key, float* out, bool required = true) {
        const JsonValue* c = v.get(key);
        if (!c) { if (required) bad(std::string("missing \"") + key + "\""); return; }
        if (c->kind != JsonValue::NUM || !std::isfinite(c->num)) { bad(std::string("\"") + key + "\" must be a number"); return; }
        *out = (float)c->num;
    }
    void real(const char* key, double* out) {
        const JsonValue* c = v.get(key);
        if (!c) bad(std::string("missing \"") + key + "\"");
        else if (c->kind != JsonValue::NUM || !std::isfinite(c->num)) bad(std::string("\"") + key + "\" must be a number");
        else *out = c->num;
    }
    void count(const char* key, int* out, bool required = true, int least = 1) {  // an integer
        const JsonValue* c = v.get(key);
        if (!c) { if (required) bad(std::string("missing \"") + key + "\""); return; }
        if (c->kind != JsonValue::NUM || c->num < least || c->num > (double)(1 << 28) || c->num != std::floor(c->num)) {
            bad(std::string("\"") + key + "\" must be a " + (least > 0 ? "positive" : "non-negative") + " integer");
            return;
        }
        *out = (int)c->num;
    }
};

bool parse_window(const JsonValue& v, const std::string& path, int* window, std::string* err) {
    Fields f{v, path, err};
    if (const JsonValue* m = f.child("mask", false)) {
        Fields g{*m, path + ".mask", err};
        g.count("size", window, false);
        f.ok = f.ok && g.ok;
    }
    return f.ok;
}

// "rot" of a mixer; `limit`: entries of the vectors that are rotated
bool parse_rotation(const JsonValue& v, const std::string& path, int limit, RotCfg* r, std::string* err) {
    Fields f{v, path, err};
    const JsonValue* c = f.child("rot", false);
    if (!c) return f.ok;
    Fields g{*c, path + ".rot", err};
    g.count("dims", &r->dims, true, 0);
    g.real("base", &r->base);
    if (g.ok && (r->dims % 2 || r->dims > limit)) g.bad("dims must be even and no more than the vectors have");
    if (g.ok && r->base <= 0.0) g.bad("base must be positive");
    const JsonValue* s = g.child("scaling", false);
    if (!s) return g.ok;
    Fields h{*s, path + ".rot.scaling", err};
    r->scaled = true;
    h.real("factor", &r->factor);
    h.real("low", &r->low);
    h.real("high", &r->high);
    h.real("original", &r->original);
    if (h.ok && !(r->factor > 0.0 && r->low > 0.0 && r->high >= r->low && r->original > 0.0)) h.bad("needs positive numbers, high no less than low");
    return g.ok && h.ok;
}

bool parse_attention(const JsonValue& v, const std::string& path, AttnCfg* a, std::string* err) {
    Fields f{v, path, err};
    f.count("heads", &a->heads);
    f.count("kv_heads", &a->kv_heads);
    f.count("dim", &a->dim);
    f.count("vdim", &a->vdim);
    f.number("scale", &a->scale);
    if (f.ok) f.ok = parse_window(v, path, &a->window, err);
    if (const JsonValue* t = f.child("q_temp", false)) {
        Fields g{*t, path + ".q_temp", err};
        g.number("coef", &a->temp_coef);
        g.count("every", &a->temp_every);
        f.ok = f.ok && g.ok;
    }
    if (f.ok && a->heads % a->kv_heads) f.bad("heads must be a multiple of kv_heads");
    return f.ok;
}

bool parse_memory(const JsonValue& v, const std::string& path, MemCfg* m, std::string* err) {
    Fields f{v, path, err};
    f.count("heads", &m->heads);
    f.count("dim", &m->dim);
    f.count("vdim", &m->vdim);
    f.number("gate_cap", &m->gate_cap);
    if (f.ok && m->gate_cap <= 0.0f) f.bad("gate_cap must be positive");
    return f.ok;
}

bool parse_ffn(const JsonValue& v, const std::string& path, FfnCfg* c, std::string* err) {
    Fields f{v, path, err};
    const JsonValue* kind = v.get("kind");
    if (!kind || kind->kind != JsonValue::STR) { f.bad("missing \"kind\""); return false; }
    if (kind->str == "dense") {
        c->kind = FfnCfg::DENSE;
        f.count("ff", &c->ff);
        return f.ok;
    }
    if (kind->str != "moe") { f.bad("unknown kind \"" + kind->str + "\""); return false; }
    c->kind = FfnCfg::MOE;
    const JsonValue *ex = f.child("expert", true), *ro = f.child("router", true);
    if (!ex || !ro) return false;
    Fields fe{*ex, path + ".expert", err}, fr{*ro, path + ".router", err};
    fe.count("ff", &c->ff);
    fr.count("experts", &c->experts);
    fr.count("top", &c->top);
    if (const JsonValue* g = fr.child("groups", false)) {
        Fields fg{*g, path + ".router.groups", err};
        fg.count("count", &c->groups);
        fg.count("keep", &c->keep);
        if (fg.ok && (c->experts % c->groups || c->keep > c->groups)) fg.bad("groups must divide the experts evenly and keep no more than there are");
        if (!fg.ok) return false;
    }
    if (!fe.ok || !fr.ok) return false;
    if (c->top > c->experts / c->groups * c->keep) { fr.bad("top exceeds the experts that may be chosen"); return false; }
    return true;
}

bool parse_latent(const JsonValue& v, const std::string& path, LatentCfg* a, std::string* err) {
    Fields f{v, path, err};
    f.count("heads", &a->heads);
    f.count("dim", &a->dim);
    f.count("rot_dim", &a->rot_dim);
    f.count("vdim", &a->vdim);
    f.count("kv_rank", &a->rank);
    f.number("scale", &a->scale);
    if (f.ok) f.ok = parse_window(v, path, &a->window, err) && parse_rotation(v, path, a->rot_dim, &a->rot, err);
    return f.ok;
}

// linear attention with a constant decay per head
bool parse_lightning(const JsonValue& v, const std::string& path, MemCfg* m, std::string* err) {
    Fields f{v, path, err};
    m->kind = MemCfg::LINEAR;
    f.count("heads", &m->heads);
    f.count("dim", &m->dim);
    f.count("vdim", &m->vdim);
    const JsonValue* d = v.get("decay");
    if (!d || d->kind != JsonValue::ARR) { f.bad("\"decay\" must be a list"); return false; }
    for (const JsonValue& x : d->arr) {
        if (x.kind != JsonValue::NUM || !(x.num >= 0.0 && x.num <= 1.0)) { f.bad("decay must lie between 0 and 1"); return false; }
        m->decay.push_back(x.num);
    }
    if (f.ok && (int)m->decay.size() != m->heads) f.bad("decay must have one number per head");
    return f.ok;
}

bool parse_differential(const JsonValue& v, const std::string& path, AttnCfg* a, std::string* err) {
    Fields f{v, path, err};
    if (!parse_attention(v, path, a, err)) return false;
    f.number("diff", &a->diff);
    a->maps = 2;
    a->gate = AttnCfg::GATE_ELEMENT;
    if (f.ok) f.ok = parse_rotation(v, path, a->dim, &a->rot, err);
    return f.ok;
}

bool parse_eps(Fields& f, float* eps) {
    if (const JsonValue* n = f.child("norm", true)) {
        Fields g{*n, "norm", f.err};
        g.number("eps", eps);
        f.ok = f.ok && g.ok;
    }
    return f.ok;
}

// Dafidra: in every layer a windowed softmax attention and a matrix memory side by side, norms on the sublayers' outputs
// only, a dense or routed feed-forward.
bool parse_dafidra(const JsonValue& root, HybridCfg* out, std::string* err) {
    Fields f{root, "config", err};
    f.count("vocab", &out->vocab);
    f.count("width", &out->width);
    f.number("residual_mult", &out->residual_mult);
    parse_eps(f, &out->eps);
    const JsonValue* layers = root.get("layers");
    if (!layers || layers->kind != JsonValue::ARR || layers->arr.empty()) { f.bad("\"layers\" must be a non-empty list"); return false; }
    for (size_t i = 0; f.ok && i < layers->arr.size(); ++i) {
        const std::string path = "layers[" + std::to_string(i) + "]";
        Fields g{layers->arr[i], path, err};
        HybridLayerCfg L;
        const JsonValue* type = layers->arr[i].get("type");
        if (!type || type->str != "parallel") { g.bad("unknown mixer type"); return false; }
        const JsonValue* mixer = g.child("mixer", true);
        if (!mixer) return false;
        Fields h{*mixer, path + ".mixer", err};
        const JsonValue *left = h.child("left", true), *right = h.child("right", true), *mlp = g.child("mlp", false);
        if (!left || !right || !g.ok) return false;
        if (!parse_attention(*left, path + ".mixer.left", &L.attn, err) || !parse_memory(*right, path + ".mixer.right", &L.mem, err)) return false;
        if (mlp && !parse_ffn(*mlp, path + ".mlp", &L.mlp, err)) return false;
        L.attn.qk_norm = L.attn.distance_bias = L.attn.sink = true;
        L.attn.gate = AttnCfg::GATE_HEAD;
        out->layers.push_back(L);
    }
    return f.ok;
}

// Kazodra: one mixer per layer (latent attention over a window, linear attention with constant decays, or differential
// attention), layer norms ahead of and behind each sublayer, a gated part of a second embedding added by every layer, and
// a run of layers that is passed several times.
bool parse_kazodra(const JsonValue& root, HybridCfg* out, std::string* err) {
    Fields f{root, "config", err};
    f.count("vocab", &out->vocab);
    f.count("width", &out->width);
    parse_eps(f, &out->eps);
    out->pre_norms = out->layer_norm = out->tied = true;
    if (const JsonValue* s = f.child("token_side", false)) {
        Fields g{*s, "token_side", err};
        g.count("dim", &out->side_dim);
        f.ok = f.ok && g.ok;
    }
    const JsonValue* layers = root.get("layers");
    if (!layers || layers->kind != JsonValue::ARR || layers->arr.empty()) { f.bad("\"layers\" must be a non-empty list"); return false; }
    for (size_t i = 0; f.ok && i < layers->arr.size(); ++i) {
        const std::string path = "layers[" + std::to_string(i) + "]", pm = path + ".mixer";
        Fields g{layers->arr[i], path, err};
        HybridLayerCfg L;
        const JsonValue *type = layers->arr[i].get("type"), *mixer = g.child("mixer", true), *mlp = g.child("mlp", false);
        if (!mixer || !g.ok) return false;
        const std::string kind = type ? type->str : "";
        bool ok;
        if (kind == "latent_attention") { L.mixer = HybridLayerCfg::LATENT; ok = parse_latent(*mixer, pm, &L.latent, err); }
        else if (kind == "lightning") { L.mixer = HybridLayerCfg::MEMORY; ok = parse_lightning(*mixer, pm, &L.mem, err); }
        else if (kind == "attention") { L.mixer = HybridLayerCfg::ATTENTION; ok = parse_differential(*mixer, pm, &L.attn, err); }
        else { g.bad("unknown mixer type"); return false; }
        if (!ok || (mlp && !parse_ffn(*mlp, path + ".mlp", &L.mlp, err))) return false;
        if (L.mlp.kind == FfnCfg::MOE) { g.bad("the feed-forward must be dense"); return false; }
        out->layers.push_back(L);
    }
    if (!f.ok) return false;
    if (const JsonValue* l = f.child("loop", false)) {
        Fields g{*l, "loop", err};
        g.count("start", &out->loop_start, true, 0);
        g.count("stop", &out->loop_stop);
        g.count("times", &out->loop_times);
        if (g.ok && (out->loop_start >= out->loop_stop || out->loop_stop > (int)out->layers.size())) g.bad("start .. stop must be a run of the layers");
        if (g.ok && (long long)(out->loop_stop - out->loop_start) * out->loop_times > 4096) g.bad("more than 4096 layer runs");
        f.ok = f.ok && g.ok;
    }
    return f.ok;
}

const ArchEntry ARCHITECTURES[] = {{"Dafidra", parse_dafidra}, {"Kazodra", parse_kazodra}};

}  // namespace

std::vector<double> rot_frequencies(const RotCfg& r) {
    const double pi = 3.14159265358979323846;
    std::vector<double> f(r.dims / 2);
    for (int i = 0; i < r.dims / 2; ++i) {
        f[i] = std::pow(r.base, -2.0 * i / r.dims);
        if (!r.scaled) continue;
        const double periods = r.original * f[i] / (2.0 * pi);  // wavelengths that fit the original context
        if (periods > r.high) continue;
        if (periods < r.low) { f[i] /= r.factor; continue; }
        const double s = r.high > r.low ? (periods - r.low) / (r.high - r.low) : 1.0;
        f[i] = (1.0 - s) * f[i] / r.factor + s * f[i];
    }
    return f;
}

std::vector<LayerRun> HybridCfg::runs() const {
    std::vector<LayerRun> out;
    const int n = (int)layers.size(), first = loop_times > 0 ? loop_start : n, behind = loop_times > 0 ? loop_stop : n;
    for (int i = 0; i < first; ++i) out.push_back({i, -1});
    for (int t = 0; t < loop_times; ++t)
        for (int i = loop_start; i < loop_stop; ++i) out.push_back({i, i == loop_start ? t : -1});
    for (int i = behind; i < n; ++i) out.push_back({i, -1});
    return out;
}

const ArchEntry* find_arch(const std::string& name) {
    for (const ArchEntry& a : ARCHITECTURES)
        if (name == a.name) return &a;
    return nullptr;
}

bool parse_hybrid_config(const std::string& text, HybridCfg* out, std::string* err) {
    JsonValue root;
    if (!JsonReader(text).parse(&root) || root.kind != JsonValue::OBJ) { *err = "config.json is not a JSON object"; return false; }
    const JsonValue* a = root.get("architecture");
    if (!a || a->kind != JsonValue::STR) { *err = "config.json names no architecture"; return false; }
    const ArchEntry* e = find_arch(a->str);
    if (!e) { *err = "unknown architecture \"" + a->str + "\""; return false; }
    out->architecture = a->str;
    return e->parse(root, out, err);
}

}  // namespace cd
