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
    void count(const char* key, int* out, bool required = true) {  // a positive integer
        const JsonValue* c = v.get(key);
        if (!c) { if (required) bad(std::string("missing \"") + key + "\""); return; }
        if (c->kind != JsonValue::NUM || c->num < 1 || c->num > (double)(1 << 28) || c->num != std::floor(c->num)) {
            bad(std::string("\"") + key + "\" must be a positive integer");
            return;
        }
        *out = (int)c->num;
    }
};

bool parse_attention(const JsonValue& v, const std::string& path, AttnCfg* a, std::string* err) {
    Fields f{v, path, err};
    f.count("heads", &a->heads);
    f.count("kv_heads", &a->kv_heads);
    f.count("dim", &a->dim);
    f.count("vdim", &a->vdim);
    f.number("scale", &a->scale);
    if (const JsonValue* m = f.child("mask", false)) {
        Fields g{*m, path + ".mask", err};
        g.count("size", &a->window, false);
        f.ok = f.ok && g.ok;
    }
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

// Dafidra: in every layer a windowed softmax attention and a matrix memory side by side, norms on the sublayers' outputs
// only, a dense or routed feed-forward.
bool parse_dafidra(const JsonValue& root, HybridCfg* out, std::string* err) {
    Fields f{root, "config", err};
    f.count("vocab", &out->vocab);
    f.count("width", &out->width);
    f.number("residual_mult", &out->residual_mult);
    if (const JsonValue* n = f.child("norm", true)) {
        Fields g{*n, "norm", err};
        g.number("eps", &out->eps);
        f.ok = f.ok && g.ok;
    }
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
        if (!parse_attention(*left, path + ".mixer.left", &L.left, err) || !parse_memory(*right, path + ".mixer.right", &L.right, err)) return false;
        if (mlp && !parse_ffn(*mlp, path + ".mlp", &L.mlp, err)) return false;
        out->layers.push_back(L);
    }
    return f.ok;
}

const ArchEntry ARCHITECTURES[] = {{"Dafidra", parse_dafidra}};

}  // namespace

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
