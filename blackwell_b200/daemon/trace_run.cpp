// Replays a trace of token ids through a config.json model and writes logits; samples nothing.
//
//   trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N
//
// Steps come from standard input, one JSON object a line:
//   {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
// Every entry's tokens continue its request through bw_decode_portion (the decode driver's slots, caches and kernels); the
// logits at the wanted places go to DIR/<step>.f32, little-endian fp32, in the order of the entries; "done <step>" follows
// on standard output.  Requests listed in "end" give their slot back.
#include <stdint.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#include <map>
#include <string>
#include <vector>

#include "../../include/blackwell_b200.h"
#include "../csrc/json.h"

namespace {

constexpr int kSlots = 4;   // requests alive at the same time

bool ints(const bw::Json* j, std::vector<int>* out) {
    if (!j || j->type != bw::Json::kArray) return false;
    for (const bw::Json& v : j->arr) {
        if (!v.is_int() || v.num < 0 || v.num > 0x7fffffff) return false;
        out->push_back((int)v.num);
    }
    return true;
}

int fail(const std::string& why) {
    fprintf(stderr, "trace_run: %s\n", why.c_str());
    return 1;
}

}  // namespace

int main(int argc, char** argv) {
    std::string model, dtype = "bfloat16", out;
    long max_tokens = 4096;
    for (int i = 1; i + 1 < argc; i += 2) {
        const std::string k = argv[i];
        if (k == "--model") model = argv[i + 1];
        else if (k == "--dtype") dtype = argv[i + 1];
        else if (k == "--out") out = argv[i + 1];
        else if (k == "--max-tokens") max_tokens = atol(argv[i + 1]);
        else return fail("unknown option " + k);
    }
    if (model.empty() || out.empty() || max_tokens < 1 || max_tokens > 0x7fffffff || (dtype != "bfloat16" && dtype != "float32"))
        return fail("usage: trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N");
    bw_decode_config cfg;
    memset(&cfg, 0, sizeof cfg);
    cfg.batch = kSlots;
    cfg.max_seq = (int)max_tokens;
    cfg.act_bits = 8;
    cfg.compute_f32 = dtype == "float32";
    cfg.weights_dir = model.c_str();
    bw_decode* eng = nullptr;
    int e = bw_decode_create(&cfg, &eng);
    if (e != 0) return fail("cannot create the engine, error " + std::to_string(e));
    bw_decode_get_config(eng, &cfg);

    std::map<std::string, int> slot_of;
    std::vector<bool> used(kSlots, false);
    std::string line, err;
    for (;;) {
        line.clear();
        int c;
        while ((c = getchar()) != EOF && c != '\n') line.push_back((char)c);
        if (line.find_first_not_of(" \t\r") == std::string::npos) {
            if (c == EOF) break;
            continue;
        }
        bw::Json j;
        if (!bw::Json::parse(line.data(), line.size(), &j, &err)) return fail(err);
        const bw::Json *step = j.get("step"), *entries = j.get("entries"), *end = j.get("end");
        if (!step || !step->is_int() || !entries || entries->type != bw::Json::kArray) return fail("a step needs 'step' and 'entries'");
        const std::string number = std::to_string((long)step->num);
        std::vector<float> logits;
        size_t rows = 0;
        for (const bw::Json& en : entries->arr) {
            const bw::Json* id = en.get("id");
            std::vector<int> tokens, want;
            if (!id || id->type != bw::Json::kString || !ints(en.get("tokens"), &tokens) || (en.get("want") && !ints(en.get("want"), &want)))
                return fail("step " + number + ": bad entry");
            if (tokens.empty()) continue;
            auto it = slot_of.find(id->str);
            if (it == slot_of.end()) {
                int s = 0;
                while (s < kSlots && used[s]) ++s;
                if (s == kSlots) return fail("step " + number + ": more than " + std::to_string(kSlots) + " requests at a time");
                used[s] = true;
                it = slot_of.emplace(id->str, s).first;
            }
            logits.resize((rows + want.size()) * (size_t)cfg.vocab);
            e = bw_decode_portion(eng, it->second, tokens.data(), (int)tokens.size(), want.data(), (int)want.size(),
                                  want.empty() ? nullptr : logits.data() + rows * (size_t)cfg.vocab, nullptr);
            int status = 0;
            if (e == 0) e = bw_device_status(&status);
            if (e != 0 || status != 0) return fail("step " + number + ": error " + std::to_string(e) + ", device status " + std::to_string(status));
            rows += want.size();
        }
        if (rows > 0) {
            const std::string path = out + "/" + number + ".f32";
            FILE* f = fopen(path.c_str(), "wb");
            if (!f || fwrite(logits.data(), 4, logits.size(), f) != logits.size() || fclose(f) != 0) return fail("cannot write " + path);
        }
        if (end)
            for (const bw::Json& id : end->arr) {
                auto it = slot_of.find(id.str);
                if (it == slot_of.end()) continue;
                bw_decode_release(eng, it->second);
                used[it->second] = false;
                slot_of.erase(it);
            }
        printf("done %s\n", number.c_str());
        fflush(stdout);
        if (c == EOF) break;
    }
    bw_decode_destroy(eng);
    return 0;
}
