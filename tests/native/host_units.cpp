// Host-side units of the model-folder backends, without a GPU: JSON, safetensors folders, block pool, sampler, and the
// scheduler's portions over a backend that only records what it is given. Prints "ok" or stops at the first failure.
#include <cmath>
#include <cstdio>
#include <cstdlib>
#include <set>
#include <string>

#include "batch_scheduler.h"
#include "block_pool.h"
#include "json_value.h"
#include "model_dir.h"
#include "token_sampler.h"

#define CHECK(c)                                                                  \
    do {                                                                          \
        if (!(c)) {                                                               \
            std::printf("failed at line %d: %s\n", __LINE__, #c);                 \
            std::exit(1);                                                         \
        }                                                                         \
    } while (0)
template <class F>
static std::string thrown(F&& f) {
    try { f(); } catch (const std::exception& e) { return e.what(); }
    return "";
}

// "Model": the logits of a token favour the sum of all tokens of the sequence so far plus one, modulo the vocabulary. It
// insists that a sequence is fed in order, once per step, within the limits it states.
struct CountingBackend : BatchedBackend {
    int portion, budget, slots, vocab = 50;
    std::vector<long> sum, len;
    std::vector<float> logits;
    int widest = 0, longest = 0, released = 0;
    CountingBackend(int portion, int budget, int slots) : portion(portion), budget(budget), slots(slots), sum(size_t(slots)), len(size_t(slots)) {}
    const float* forward_multi(const int32_t* tok, const int32_t* seq, const int32_t* pos, int n) override {
        CHECK(n >= 1 && n <= slots);
        logits.assign(size_t(n) * size_t(vocab), 0.f);
        for (int i = 0; i < n; i++) {
            CHECK(pos[i] == len[size_t(seq[i])]);
            sum[size_t(seq[i])] += tok[i];
            len[size_t(seq[i])]++;
            logits[size_t(i * vocab) + size_t((sum[size_t(seq[i])] + 1) % vocab)] = 1.f;
        }
        return logits.data();
    }
    const float* forward_step(const StepEntry* e, int n, int nv) override {
        if (portion == 1) return BatchedBackend::forward_step(e, n, nv);
        std::set<int> seen;
        int total = 0, rows = 0;
        for (int i = 0; i < n; i++) { CHECK(seen.insert(e[i].seq_id).second); total += e[i].n_tokens; rows += e[i].n_want; longest = std::max(longest, e[i].n_tokens); }
        CHECK(total <= budget);
        widest = std::max(widest, total);
        std::vector<float> out(size_t(rows) * size_t(vocab), 0.f);
        int r = 0;
        for (int i = 0; i < n; i++) {
            const size_t s = size_t(e[i].seq_id);
            CHECK(e[i].pos0 == len[s] && e[i].n_tokens >= 1 && e[i].n_tokens <= portion);
            for (int t = 0; t < e[i].n_tokens; t++) {
                sum[s] += e[i].tokens[t];
                len[s]++;
                for (int w = 0; w < e[i].n_want; w++)
                    if (e[i].want[w] == t) out[size_t(r++) * size_t(vocab) + size_t((sum[s] + 1) % vocab)] = 1.f;
            }
        }
        CHECK(r == rows);
        logits = out;
        return rows ? logits.data() : nullptr;
    }
    void release_sequence(int s) override { sum[size_t(s)] = len[size_t(s)] = 0; released++; }
    int max_seqs() const override { return slots; }
    int n_ctx_per_seq() const override { return 400; }
    int max_portion() const override { return portion; }
    int max_step_tokens() const override { return budget; }
};
using Scheduler = BasicBatchScheduler<TokenSampler, TokenSamplerParams>;

static std::vector<std::vector<int32_t>> serve(CountingBackend& b, long long* steps) {
    Scheduler s(b, b.vocab);
    std::vector<int> ids;
    for (int r = 0; r < 6; r++) {
        Scheduler::Request q;
        for (int i = 0; i < 1 + 37 * r % 101; i++) q.prompt.push_back((i * 7 + r) % b.vocab);
        q.max_tokens = 3 + r;
        ids.push_back(s.submit(q));
        if (r % 2) s.step();
    }
    s.run();
    std::vector<std::vector<int32_t>> out;
    for (int id : ids) { CHECK(std::string(s.result(id).finish) == "length"); out.push_back(s.result(id).tokens); }
    *steps = s.steps();
    CHECK(b.released == 6);
    return out;
}

int main(int argc, char** argv) {
    CHECK(argc == 3);
    const Json j = Json::parse(" {\"a\": [1, -2.5e1, true, null, \"x\\n\\u00e9\"], \"b\": {}} ");
    CHECK(j.at("a").items().size() == 5 && j.at("a").items()[1].number() == -25 && j.at("a").items()[4].str() == "x\n\xc3\xa9" && j.at("b").is_object());
    CHECK(thrown([] { Json::parse("{\"a\": }"); }) != "" && thrown([] { Json::parse("[1] 2"); }) != "" && thrown([] { Json::parse("[1"); }) != "");
    CHECK(thrown([&] { j.at("c"); }).find("\"c\" is missing") != std::string::npos && thrown([&] { j.at("a").items()[1].str(); }) != "");

    ModelDir dir(argv[1]);
    CHECK(dir.config().at("architecture").str() == "Besudra" && dir.has("embed") && !dir.has("nothing"));
    CHECK(thrown([&] { dir.tensor("embed", {1, 2}); }).find("shape") != std::string::npos && thrown([&] { dir.tensor("nothing"); }) != "");
    const std::vector<float> norm = tensor_f32(dir.tensor("final.norm"));
    CHECK(int64_t(norm.size()) == dir.config().at("width").integer() && std::fabs(norm[0]) < 10.f);
    CHECK(thrown([&] { ModelDir bad(argv[2]); }).find("outside the file") != std::string::npos);

    BlockPool pool(5, 2, 8);
    pool.ensure(0, 0, 1);
    pool.ensure(1, 3, 4);
    pool.ensure(0, 0, 2);
    CHECK(pool.free_blocks() == 0 && thrown([&] { pool.ensure(1, 3, 5); }) == "context window exceeded" && thrown([&] { pool.ensure(1, 0, 8); }) != "");
    std::set<int> held = {pool.row(0)[0], pool.row(0)[1], pool.row(0)[2], pool.row(1)[3], pool.row(1)[4]};
    CHECK(held.size() == 5);
    const int freed = pool.row(0)[1];
    pool.release(0, 1, 2);
    pool.ensure(1, 7, 7);
    CHECK(pool.row(1)[7] == freed && pool.row(0)[1] == -1);
    pool.release(1);
    CHECK(pool.free_blocks() == 3);

    {  // sampler: greedy takes the lower id of a tie, penalties and limits apply, a seed repeats
        float l[4] = {0, 2, 2, 1};
        CHECK(TokenSampler({}, 4).sample(l, {}) == 1);
        TokenSamplerParams p;
        p.repeat_penalty = 4;
        CHECK(TokenSampler(p, 4).sample(l, {1}) == 2);
        p = {};
        p.temperature = 1;
        p.top_k = 1;
        float m[4] = {0, 1, 5, 1};
        CHECK(TokenSampler(p, 4).sample(m, {}) == 2);
        p.top_k = 0;
        p.top_p = 0.5f;
        CHECK(TokenSampler(p, 4).sample(m, {}) == 2);
        p.top_p = 1;
        p.temperature = 5;
        TokenSampler a(p, 4), b(p, 4);
        std::set<int> kinds;
        for (int i = 0; i < 200; i++) { const int x = a.sample(m, {}); CHECK(x == b.sample(m, {})); kinds.insert(x); }
        CHECK(kinds.size() == 4);
    }

    long long single = 0, portions = 0;
    CountingBackend one(1, 3, 3), many(16, 20, 3);
    const auto a = serve(one, &single), b = serve(many, &portions);
    CHECK(a == b && portions < single / 3 && many.widest > 3 && many.longest > 1);
    std::printf("ok\n");
}
