// Command line over the model registry:
//   ingot_models list
//   ingot_models info     --model DIR
//   ingot_models generate --model DIR --prompt-ids 1,2,3 [--prompt-ids ...] [--max-new N] [sampling options]
//   ingot_models trace    --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N     (steps on standard input)
// Tokens are ids: these model folders carry no tokenizer.
#include <cstdio>
#include <cstdlib>
#include <cstring>
#include <iostream>
#include <map>
#include <string>
#include <vector>

#include "batch_scheduler.h"
#include "model_registry.h"
#include "token_sampler.h"

namespace {

struct Args {
    std::vector<std::pair<std::string, std::string>> options;
    const std::string* find(const std::string& key) const {
        for (const auto& o : options)
            if (o.first == key) return &o.second;
        return nullptr;
    }
    std::string need(const std::string& key) const {
        const std::string* v = find(key);
        if (!v) throw std::runtime_error("missing option " + key);
        return *v;
    }
    double number(const std::string& key, double fallback) const {
        const std::string* v = find(key);
        if (!v) return fallback;
        char* end = nullptr;
        const double d = std::strtod(v->c_str(), &end);
        if (v->empty() || *end) throw std::runtime_error("option " + key + " needs a number");
        return d;
    }
    bool f32() const {
        const std::string* v = find("--dtype");
        if (!v || *v == "bfloat16") return false;
        if (*v == "float32") return true;
        throw std::runtime_error("--dtype is bfloat16 or float32");
    }
};

// Replays a trace: every line of standard input is one step {"step", "entries": [{"id", "tokens", "want"}], "end": [ids]}.
// A step's wanted logits go to OUT/<step>.f32; "done <step>" follows on standard output. Requests are named; the engine's
// sequence slots are given out at a request's first entry and come back when it ends.
int trace(const Args& a) {
    EngineOptions opt;
    opt.f32 = a.f32();
    opt.max_seqs = int(a.number("--max-seqs", 4));
    opt.max_tokens = int(a.number("--max-tokens", 0));
    if (opt.max_tokens < 1) throw std::runtime_error("--max-tokens needs a positive number");
    const std::string out = a.need("--out");
    auto backend = open_model(a.need("--model"), opt);
    const int n_vocab = backend->n_vocab();
    struct Live { int seq; int pos; };
    std::map<std::string, Live> live;
    std::vector<int> free_seqs;
    for (int s = opt.max_seqs - 1; s >= 0; s--) free_seqs.push_back(s);

    std::string line;
    while (std::getline(std::cin, line)) {
        if (line.find_first_not_of(" \t\r") == std::string::npos) continue;
        const Json j = Json::parse(line);
        const long long step = j.at("step").integer();
        const auto& items = j.at("entries").items();
        std::vector<std::vector<int32_t>> tokens(items.size()), want(items.size());
        std::vector<StepEntry> entries;
        std::vector<Live*> who;
        size_t rows = 0;
        for (size_t i = 0; i < items.size(); i++) {
            const std::string& id = items[i].at("id").str();
            for (const Json& t : items[i].at("tokens").items()) tokens[i].push_back(int32_t(t.integer()));
            for (const Json& w : items[i].at("want").items()) want[i].push_back(int32_t(w.integer()));
            auto it = live.find(id);
            if (it == live.end()) {
                if (free_seqs.empty()) throw std::runtime_error("trace: more live requests than sequence slots");
                it = live.emplace(id, Live{free_seqs.back(), 0}).first;
                free_seqs.pop_back();
            }
            if (tokens[i].empty()) continue;
            entries.push_back(StepEntry{it->second.seq, it->second.pos, tokens[i].data(), int32_t(tokens[i].size()), want[i].data(), int32_t(want[i].size())});
            who.push_back(&it->second);
            rows += want[i].size();
        }
        const float* logits = entries.empty() ? nullptr : backend->forward_step(entries.data(), int(entries.size()), n_vocab);
        for (size_t i = 0; i < entries.size(); i++) who[i]->pos += entries[i].n_tokens;
        if (rows) {
            const std::string path = out + "/" + std::to_string(step) + ".f32";
            FILE* f = std::fopen(path.c_str(), "wb");
            if (!f) throw std::runtime_error("trace: cannot write " + path);
            const size_t n = rows * size_t(n_vocab);
            const bool ok = std::fwrite(logits, sizeof(float), n, f) == n;
            if (std::fclose(f) != 0 || !ok) throw std::runtime_error("trace: cannot write " + path);
        }
        for (const Json& e : j.at("end").items()) {
            auto it = live.find(e.str());
            if (it == live.end()) continue;
            backend->release_sequence(it->second.seq);
            free_seqs.push_back(it->second.seq);
            live.erase(it);
        }
        std::printf("done %lld\n", step);
        std::fflush(stdout);
    }
    return 0;
}

int generate(const Args& a) {
    EngineOptions opt;
    opt.f32 = a.f32();
    std::vector<std::vector<int32_t>> prompts;
    for (const auto& o : a.options)
        if (o.first == "--prompt-ids") {
            prompts.emplace_back();
            for (size_t at = 0; at < o.second.size();) {
                char* end = nullptr;
                const char* begin = o.second.c_str() + at;
                prompts.back().push_back(int32_t(std::strtol(begin, &end, 10)));
                if (end == begin || (*end && *end != ',')) throw std::runtime_error("--prompt-ids takes ids separated by commas");
                at += size_t(end - begin) + 1;
            }
        }
    if (prompts.empty()) throw std::runtime_error("missing option --prompt-ids");
    opt.max_seqs = int(a.number("--max-seqs", 8));
    opt.max_tokens = int(a.number("--max-tokens", 4096));
    opt.max_step_tokens = int(a.number("--max-step-tokens", 2048));
    auto backend = open_model(a.need("--model"), opt);
    BasicBatchScheduler<TokenSampler, TokenSamplerParams> sched(*backend, backend->n_vocab());
    const int stop = int(a.number("--stop-id", -1));
    std::vector<int> ids;
    for (auto& p : prompts) {
        BasicBatchScheduler<TokenSampler, TokenSamplerParams>::Request r;
        r.prompt = p;
        r.max_tokens = int(a.number("--max-new", 32));
        r.sampling.temperature = float(a.number("--temp", 0));
        r.sampling.top_k = int(a.number("--top-k", 0));
        r.sampling.top_p = float(a.number("--top-p", 1));
        r.sampling.repeat_penalty = float(a.number("--repeat-penalty", 1));
        r.sampling.seed = uint64_t(a.number("--seed", 0));
        if (stop >= 0) r.is_stop = [stop](int32_t t) { return t == stop; };
        ids.push_back(sched.submit(std::move(r)));
    }
    sched.run();
    for (int id : ids) {
        const auto& res = sched.result(id);
        for (size_t i = 0; i < res.tokens.size(); i++) std::printf("%s%d", i ? "," : "", res.tokens[i]);
        std::printf("  # %s\n", res.finish ? res.finish : "");
    }
    return 0;
}

int usage() {
    std::fprintf(stderr,
                 "usage: ingot_models list\n"
                 "       ingot_models info --model DIR [--dtype bfloat16|float32]\n"
                 "       ingot_models generate --model DIR --prompt-ids 1,2,3 [--prompt-ids ...] [--max-new N] [--stop-id T]\n"
                 "                    [--temp T --top-k K --top-p P --repeat-penalty R --seed S] [--dtype bfloat16|float32]\n"
                 "                    [--max-seqs N --max-tokens N --max-step-tokens N]\n"
                 "       ingot_models trace --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N [--max-seqs N]\n");
    return 2;
}

}  // namespace

int main(int argc, char** argv) {
    try {
        if (argc < 2) return usage();
        const std::string verb = argv[1];
        Args a;
        for (int i = 2; i < argc; i++) {
            const std::string key = argv[i];
            if (key.rfind("--", 0) != 0 || i + 1 >= argc) return usage();
            a.options.emplace_back(key, argv[++i]);
        }
        if (verb == "list") {
            for (const std::string& n : registered_architectures()) std::printf("%s\n", n.c_str());
            return 0;
        }
        if (verb == "info") {
            EngineOptions opt;
            opt.f32 = a.f32();
            opt.max_tokens = 64;
            opt.max_seqs = 1;
            auto b = open_model(a.need("--model"), opt);
            std::printf("%s, %.3f GB of weights read per step\n", b->describe().c_str(), double(b->weight_bytes()) / 1e9);
            return 0;
        }
        if (verb == "generate") return generate(a);
        if (verb == "trace") return trace(a);
        return usage();
    } catch (const std::exception& e) {
        std::fprintf(stderr, "ingot_models: %s\n", e.what());
        return 1;
    }
}
