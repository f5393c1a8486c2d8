// `trace_run` - replays a trace of requests through a model folder, step by step, and writes the logits it asks for.
//
//   trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N
//
// Standard input: one JSON object a line, {"step": 0, "entries": [{"id": "a", "tokens": [..], "want": [..]}], "end": [..]}:
// the next tokens of each request, the places among them whose logits are wanted, and the requests that end after the
// step.  A step with wanted places writes OUT/<step>.f32 ([wanted][vocab], little-endian fp32, in the order asked for);
// every step prints `done <step>`.  One request is live at a time: it holds the model's cache and state until it ends.
#include <cstdio>
#include <cstring>
#include <iostream>
#include <string>
#include <vector>

#include "../../include/cuda_decode.h"
#include "json.h"

namespace {

[[noreturn]] void die(const std::string& msg) {
    fprintf(stderr, "trace_run: %s\n", msg.c_str());
    exit(1);
}
void check(int rc, cd_model* m) {
    if (rc) die(cd_last_error(m));
}
size_t count(const cd::JsonValue& v, const char* what) {
    if (v.kind != cd::JsonValue::NUM || v.num < 0 || v.num > 4294967295.0 || v.num != (double)(size_t)v.num) die(std::string("bad ") + what);
    return (size_t)v.num;
}

}  // namespace

int main(int argc, char** argv) {
    std::string dir, out_dir, dtype = "bfloat16";
    size_t max_tokens = 0;
    for (int i = 1; i < argc; i += 2) {
        const std::string k = argv[i];
        if (i + 1 >= argc) die("missing value of " + k);
        if (k == "--model") dir = argv[i + 1];
        else if (k == "--dtype") dtype = argv[i + 1];
        else if (k == "--out") out_dir = argv[i + 1];
        else if (k == "--max-tokens") max_tokens = (size_t)strtoull(argv[i + 1], nullptr, 10);
        else die("unknown argument " + k);
    }
    if (dir.empty() || out_dir.empty()) die("usage: trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N");
    cd_options opts;
    memset(&opts, 0, sizeof opts);
    opts.device = -1;
    opts.use_graph = 1;
    if (dtype == "bfloat16") opts.weight_dtype = CD_DTYPE_BF16;
    else if (dtype == "float32") opts.weight_dtype = CD_DTYPE_F32;
    else die("--dtype must be bfloat16 or float32");
    cd_model* m = nullptr;
    check(cd_model_create_from_dir(dir.c_str(), max_tokens, &opts, &m), nullptr);
    cd_config cfg;
    cd_model_get_config(m, &cfg, nullptr, nullptr);

    std::string line, live;
    bool have_live = false;
    while (std::getline(std::cin, line)) {
        if (line.find_first_not_of(" \t\r") == std::string::npos) continue;
        cd::JsonValue root;
        if (!cd::JsonReader(line).parse(&root)) die("malformed input line");
        const cd::JsonValue *step = root.get("step"), *entries = root.get("entries"), *end = root.get("end");
        if (!step || !entries || entries->kind != cd::JsonValue::ARR) die("a step needs \"step\" and \"entries\"");
        std::vector<float> logits;
        for (const auto& e : entries->arr) {
            const cd::JsonValue *id = e.get("id"), *toks = e.get("tokens"), *want = e.get("want");
            if (!id || !toks || toks->kind != cd::JsonValue::ARR) die("an entry needs \"id\" and \"tokens\"");
            if (!have_live || live != id->str) {
                if (have_live) die("request " + id->str + " begins before " + live + " has ended");
                live = id->str;
                have_live = true;
                check(cd_set_len(m, 0), m);
            }
            std::vector<uint32_t> ids;
            std::vector<size_t> places;
            for (const auto& t : toks->arr) ids.push_back((uint32_t)count(t, "token id"));
            if (want)
                for (const auto& w : want->arr) places.push_back(count(w, "wanted place"));
            if (ids.empty()) {
                if (!places.empty()) die("places wanted of an empty portion");
                continue;
            }
            const size_t at = logits.size();
            logits.resize(at + places.size() * (size_t)cfg.vocab);
            check(cd_prefill_logits(m, ids.data(), ids.size(), places.data(), places.size(), 0.0f, logits.data() + at), m);
        }
        if (end)
            for (const auto& id : end->arr)
                if (have_live && id.str == live) {  // its cache rows and state are free for the next one
                    have_live = false;
                    check(cd_set_len(m, 0), m);
                }
        const long long n = (long long)count(*step, "step number");
        if (!logits.empty()) {
            const std::string path = out_dir + "/" + std::to_string(n) + ".f32";
            FILE* f = fopen(path.c_str(), "wb");
            if (!f || fwrite(logits.data(), 4, logits.size(), f) != logits.size() || fclose(f) != 0) die("cannot write " + path);
        }
        printf("done %lld\n", n);
        fflush(stdout);
    }
    cd_model_destroy(m);
    return 0;
}
