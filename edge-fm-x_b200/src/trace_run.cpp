// Trace runner: replays given token ids through a model's batched steps and writes the logits asked for.  Nothing is
// sampled.  Steps arrive on standard input, one JSON object a line:
//     {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [1]}], "end": ["b"]}
// entries: each request's next tokens and the places among them whose logits are wanted; end: requests that are finished
// after the step.  A step's logits go to <out>/<step>.f32 ([wanted, vocab] little-endian fp32) when something is wanted;
// "done <step>" is printed after every step.
#include <edge-fm/core.h>

#include <cstdio>
#include <cstring>
#include <iostream>
#include <string>

#include "engine/config.h"
#include "engine/standard_engine.h"

using namespace edge_fm;

namespace {

int usage(const char* why) {
    std::fprintf(stderr, "trace_run: %s\nusage: trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N\n", why);
    return 2;
}

json::Value str(const std::string& s) { json::Value v; v.type = json::Value::String; v.str = s; return v; }
json::Value num(int64_t n) { json::Value v; v.type = json::Value::Number; v.is_int = true; v.inum = n; v.num = (double)n; return v; }

std::vector<int32_t> ints(const json::Value* v) {
    std::vector<int32_t> out;
    if (v != nullptr)
        for (const json::Value& e : v->arr) out.push_back((int32_t)e.inum);
    return out;
}

}  // namespace

int main(int argc, char** argv) {
    std::string model, dtype = "bfloat16", out;
    long max_tokens = 0;
    for (int i = 1; i < argc; i += 2) {
        const std::string k = argv[i];
        if (i + 1 >= argc) return usage(("no value for " + k).c_str());
        if (k == "--model") model = argv[i + 1];
        else if (k == "--dtype") dtype = argv[i + 1];
        else if (k == "--out") out = argv[i + 1];
        else if (k == "--max-tokens") max_tokens = std::atol(argv[i + 1]);
        else return usage(("unknown option " + k).c_str());
    }
    if (model.empty() || out.empty() || max_tokens <= 0) return usage("--model, --out and a positive --max-tokens are required");
    if (dtype != "bfloat16" && dtype != "float32") return usage("--dtype must be bfloat16 or float32");
    const std::string engine_dtype = dtype == "float32" ? "fp32" : "bf16";
    try {
        json::Value cfg, runtime, cache, none;
        none.type = json::Value::Array;
        runtime.set("device", str("cuda"));
        runtime.set("compute_dtype", str(engine_dtype));
        cache.set("dtype", str(engine_dtype));
        cache.set("attention_type", str("gqa"));
        cache.set("requests", none);
        cache.set("pool_tokens", num(max_tokens));
        cache.set("max_live_requests", num(4));
        cfg.set("prefill_model_path", str(model));
        cfg.set("runtime", runtime);
        cfg.set("kvcache", cache);
        StandardEngine engine(EngineConfig(cfg, "."));
        std::string line;
        while (std::getline(std::cin, line)) {
            if (line.find_first_not_of(" \t\r\n") == std::string::npos) continue;
            const json::Value step = json::parse(line);
            const long long id = (long long)step.get_int("step", 0);
            std::vector<StepEntry> entries;
            size_t wanted = 0;
            const json::Value* list = step.find("entries");
            if (list != nullptr)
                for (const json::Value& e : list->arr) {
                    entries.push_back(StepEntry{e.get_string("id", ""), ints(e.find("tokens")), ints(e.find("want"))});
                    wanted += entries.back().want.size();
                }
            std::vector<float> logits;
            if (!entries.empty()) logits = engine.step(entries);
            const json::Value* end = step.find("end");
            if (end != nullptr)
                for (const json::Value& e : end->arr) engine.finish(e.str);
            if (wanted > 0) {
                const std::string path = out + "/" + std::to_string(id) + ".f32";
                std::FILE* f = std::fopen(path.c_str(), "wb");
                const bool ok = f != nullptr && std::fwrite(logits.data(), sizeof(float), logits.size(), f) == logits.size();
                if (f == nullptr || std::fclose(f) != 0 || !ok) throw std::runtime_error("writing " + path + " failed");
            }
            std::printf("done %lld\n", id);
            std::fflush(stdout);
        }
    } catch (const std::exception& e) {
        std::fprintf(stderr, "trace_run: %s\n", e.what());
        return 1;
    }
    return 0;
}
