// C interface over the model registry, the step function and the scheduler, for the tests, bench.py and other languages.
// Every call returns 0 (or a handle / a count) and leaves its message in ingot_models_last_error() otherwise.
#include <cstdint>
#include <memory>
#include <string>
#include <vector>

#include "batch_scheduler.h"
#include "model_registry.h"
#include "token_sampler.h"

static thread_local std::string g_models_error;

struct ingot_model {
    std::unique_ptr<ModelBackend> backend;
    std::vector<float> residuals;
};

template <class F>
static int guarded(F&& f) {
    try {
        f();
        return 0;
    } catch (const std::exception& e) {
        g_models_error = e.what();
        return -1;
    }
}

extern "C" {

const char* ingot_models_last_error() { return g_models_error.c_str(); }

// f32: 0 bf16 form, 1 32-bit form. max_step_tokens 0: max_tokens. Null on failure.
ingot_model* ingot_model_open(const char* dir, int f32, int max_tokens, int max_seqs, int max_step_tokens) {
    ingot_model* m = nullptr;
    guarded([&] {
        EngineOptions o;
        o.f32 = f32 != 0;
        o.max_tokens = max_tokens;
        o.max_seqs = max_seqs;
        o.max_step_tokens = max_step_tokens;
        auto fresh = std::make_unique<ingot_model>();
        fresh->backend = open_model(dir, o);
        m = fresh.release();
    });
    return m;
}
void ingot_model_close(ingot_model* m) { delete m; }
int ingot_model_vocab(const ingot_model* m) { return m->backend->n_vocab(); }
long long ingot_model_weight_bytes(const ingot_model* m) { return (long long)m->backend->weight_bytes(); }
float ingot_model_last_step_ms(const ingot_model* m) { return m->backend->last_step_ms(); }

// One step: n portions; tokens and want hold the portions' tokens and wanted places back to back. logits_out (may be null)
// receives the wanted rows [total wanted][vocab].
int ingot_model_step(ingot_model* m, int n, const int32_t* seq_ids, const int32_t* pos0, const int32_t* n_tokens, const int32_t* tokens,
                     const int32_t* n_want, const int32_t* want, float* logits_out) {
    return guarded([&] {
        std::vector<StepEntry> e;
        size_t rows = 0;
        for (int i = 0; i < n; i++) {
            e.push_back(StepEntry{seq_ids[i], pos0[i], tokens, n_tokens[i], want, n_want[i]});
            tokens += n_tokens[i];
            want += n_want[i];
            rows += size_t(n_want[i]);
        }
        const float* logits = m->backend->forward_step(e.data(), n, m->backend->n_vocab());
        if (logits_out && logits) std::copy(logits, logits + rows * size_t(m->backend->n_vocab()), logits_out);
    });
}
int ingot_model_release(ingot_model* m, int seq_id) {
    return guarded([&] { m->backend->release_sequence(seq_id); });
}

// Residual stream after every layer of the steps that follow: on != 0 starts collecting, ingot_model_residuals copies up to
// n floats of what was collected (returns their total number) and clears it.
void ingot_model_tap(ingot_model* m, int on) { m->backend->tap_residuals(on ? &m->residuals : nullptr); }
long long ingot_model_residuals(ingot_model* m, float* out, long long n) {
    const long long total = (long long)m->residuals.size();
    std::copy(m->residuals.begin(), m->residuals.begin() + std::min(n, total), out);
    m->residuals.clear();
    return total;
}

// n_req requests through the scheduler. prompts back to back; arrival_step may be null (all at the start); sampling: null for
// greedy, else {temperature, top_k, top_p, repeat_penalty, repeat_last_n, seed}; stop_token -1: none. out_ids [n_req][max_out],
// out_counts [n_req]; stats (may be null): backend steps and tokens they carried.
int ingot_model_generate(ingot_model* m, const int32_t* prompts, const int32_t* prompt_lens, const int32_t* max_tokens, const int32_t* arrival_step,
                         int n_req, int stop_token, const double* sampling, int32_t* out_ids, int max_out, int32_t* out_counts, long long* stats) {
    return guarded([&] {
        BasicBatchScheduler<TokenSampler, TokenSamplerParams> sched(*m->backend, m->backend->n_vocab());
        std::vector<int> id(static_cast<size_t>(n_req), -1);
        int submitted = 0;
        for (long long step = 0;; step++) {
            const int32_t* p = prompts;
            for (int r = 0; r < n_req; p += prompt_lens[r], r++) {
                if (id[size_t(r)] >= 0 || (arrival_step && arrival_step[r] > step)) continue;
                BasicBatchScheduler<TokenSampler, TokenSamplerParams>::Request q;
                q.prompt.assign(p, p + prompt_lens[r]);
                q.max_tokens = max_tokens[r];
                if (stop_token >= 0) q.is_stop = [stop_token](int32_t t) { return t == stop_token; };
                if (sampling) {
                    q.sampling.temperature = float(sampling[0]);
                    q.sampling.top_k = int(sampling[1]);
                    q.sampling.top_p = float(sampling[2]);
                    q.sampling.repeat_penalty = float(sampling[3]);
                    q.sampling.repeat_last_n = int(sampling[4]);
                    q.sampling.seed = uint64_t(sampling[5]);
                }
                id[size_t(r)] = sched.submit(std::move(q));
                submitted++;
            }
            if (!sched.step() && submitted == n_req) break;
        }
        for (int r = 0; r < n_req; r++) {
            const auto& res = sched.result(id[size_t(r)]);
            if (int(res.tokens.size()) > max_out) throw std::runtime_error("generate: reply longer than the output rows");
            out_counts[r] = int32_t(res.tokens.size());
            std::copy(res.tokens.begin(), res.tokens.end(), out_ids + size_t(r) * size_t(max_out));
        }
        if (stats) { stats[0] = sched.steps(); stats[1] = sched.rows(); }
    });
}

}  // extern "C"
