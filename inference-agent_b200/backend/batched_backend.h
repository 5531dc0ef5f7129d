// Batched extension of the compute boundary: one forward step for many independent sequences.
//
// This interface has no counterpart in the reference, whose Backend runs one sequence (one token or one chunk
// of it per call) and whose server handles one connection at a time. It exists so that the paged KV cache and
// the multi-sequence decode kernel of libingot_cuda.so (ingot_attn_decode with n_seq > 1, ingot_rope_kv_append
// with per-token positions and sequence ids) have a caller that a serving loop can drive: continuous batching
// is "call forward_multi with whatever sequences have a token ready".
//
// Semantics follow the single-sequence Backend: a sequence's cache is a pure function of (sequence, position),
// positions may be revisited, and the returned logits live in writable host memory owned by the backend until
// the next call.
#pragma once

#include <cstdint>
#include <stdexcept>
#include <vector>

// The next tokens of one sequence in a step, and the places among them whose logits are asked for.
struct StepEntry {
    int32_t seq_id = 0;
    int32_t pos0 = 0;                  // position of tokens[0]
    const int32_t* tokens = nullptr;
    int32_t n_tokens = 0;
    const int32_t* want = nullptr;     // indices into tokens, ascending
    int32_t n_want = 0;
};

class BatchedBackend {
public:
    virtual ~BatchedBackend() = default;
    // One token for each of n DIFFERENT sequences: tokens[i] of sequence seq_ids[i] (0 <= id < max_seqs()) sits at
    // position positions[i], is written to that sequence's cache and attends to its keys 0..positions[i].
    // Returns n rows of n_vocab logits, row i for tokens[i]. Throws std::runtime_error with the reference's
    // messages for a bad token id ("token id out of range") or position ("context window exceeded"), and for a
    // repeated or out-of-range sequence id.
    virtual const float* forward_multi(const int32_t* tokens, const int32_t* seq_ids, const int32_t* positions, int n) = 0;
    // The general step: one batch of portions of n DIFFERENT sequences, of one or more tokens each (portions of prompts beside
    // single decoded tokens). Returns the wanted rows of n_vocab logits in the order of the entries and of their `want` (writable
    // host memory, valid until the next call), or null if nothing is wanted. This default feeds a backend that takes one token
    // of a sequence per call; such a backend needs no portions, so max_portion() tells callers not to make any.
    virtual const float* forward_step(const StepEntry* entries, int n, int n_vocab) {
        int longest = 0;
        for (int i = 0; i < n; i++) longest = entries[i].n_tokens > longest ? entries[i].n_tokens : longest;
        size_t total = 0;
        std::vector<size_t> first(static_cast<size_t>(n));
        for (int i = 0; i < n; i++) { first[size_t(i)] = total; total += size_t(entries[i].n_want); }
        step_logits_.resize(total * size_t(n_vocab));
        for (int t = 0; t < longest; t++) {
            std::vector<int32_t> tok, seq, pos;
            std::vector<int> src;
            for (int i = 0; i < n; i++) {
                if (t >= entries[i].n_tokens) continue;
                tok.push_back(entries[i].tokens[t]);
                seq.push_back(entries[i].seq_id);
                pos.push_back(entries[i].pos0 + t);
                src.push_back(i);
            }
            const float* rows = forward_multi(tok.data(), seq.data(), pos.data(), int(tok.size()));
            for (size_t r = 0; r < src.size(); r++) {
                const StepEntry& e = entries[src[r]];
                for (int w = 0; w < e.n_want; w++)
                    if (e.want[w] == t) {
                        const float* from = rows + r * size_t(n_vocab);
                        float* to = step_logits_.data() + (first[size_t(src[r])] + size_t(w)) * size_t(n_vocab);
                        for (int v = 0; v < n_vocab; v++) to[v] = from[v];
                    }
            }
        }
        return total ? step_logits_.data() : nullptr;
    }
    // Most tokens of one sequence that a step may carry with profit (1: single tokens only), and most tokens of a step.
    virtual int max_portion() const { return 1; }
    virtual int max_step_tokens() const { return max_seqs(); }
    // Gives a sequence's cache blocks back to the pool (its id can then serve a new request).
    virtual void release_sequence(int seq_id) = 0;
    virtual int max_seqs() const = 0;
    virtual int n_ctx_per_seq() const = 0;

private:
    std::vector<float> step_logits_;  // of the default forward_step
};
