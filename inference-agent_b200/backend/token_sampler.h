// Token sampling for models that do not come with the reference's sources: repetition penalty over the last tokens,
// temperature, top-k, top-p, a seeded generator per request. temperature 0 is greedy (ties to the lower id). The
// interface is the one BasicBatchScheduler expects.
#pragma once

#include <algorithm>
#include <cmath>
#include <cstdint>
#include <numeric>
#include <random>
#include <vector>

struct TokenSamplerParams {
    float temperature = 0.0f;
    int top_k = 0;               // 0: no limit
    float top_p = 1.0f;
    float repeat_penalty = 1.0f;
    int repeat_last_n = 64;
    uint64_t seed = 0;
};

class TokenSampler {
public:
    TokenSampler(const TokenSamplerParams& p, int n_vocab) : p_(p), n_vocab_(n_vocab), rng_(p.seed) {}

    // logits [n_vocab] may be edited in place.
    int32_t sample(float* logits, const std::vector<int32_t>& history) {
        if (p_.repeat_penalty != 1.0f) {
            const size_t n = history.size(), from = p_.repeat_last_n > 0 && n > size_t(p_.repeat_last_n) ? n - size_t(p_.repeat_last_n) : 0;
            std::vector<int32_t> seen(history.begin() + long(from), history.end());
            std::sort(seen.begin(), seen.end());
            seen.erase(std::unique(seen.begin(), seen.end()), seen.end());
            for (int32_t t : seen)
                if (t >= 0 && t < n_vocab_) logits[t] = logits[t] > 0 ? logits[t] / p_.repeat_penalty : logits[t] * p_.repeat_penalty;
        }
        if (p_.temperature <= 0.0f) return int32_t(std::max_element(logits, logits + n_vocab_) - logits);
        order_.resize(size_t(n_vocab_));
        std::iota(order_.begin(), order_.end(), 0);
        const size_t k = p_.top_k > 0 ? std::min(size_t(p_.top_k), order_.size()) : order_.size();
        std::partial_sort(order_.begin(), order_.begin() + long(k), order_.end(),
                          [&](int32_t a, int32_t b) { return logits[a] != logits[b] ? logits[a] > logits[b] : a < b; });
        prob_.resize(k);
        double sum = 0;
        for (size_t i = 0; i < k; i++) sum += prob_[i] = std::exp(double(logits[order_[i]] - logits[order_[0]]) / double(p_.temperature));
        size_t keep = k;
        if (p_.top_p < 1.0f) {
            double c = 0;
            for (keep = 0; keep < k && c < double(p_.top_p) * sum; keep++) c += prob_[keep];
            keep = std::max<size_t>(keep, 1);
            sum = c > 0 ? c : prob_[0];
        }
        double u = std::uniform_real_distribution<double>(0.0, sum)(rng_);
        for (size_t i = 0; i < keep; i++)
            if ((u -= prob_[i]) < 0) return order_[i];
        return order_[keep - 1];
    }

private:
    TokenSamplerParams p_;
    int n_vocab_;
    std::mt19937_64 rng_;
    std::vector<int32_t> order_;
    std::vector<double> prob_;
};
