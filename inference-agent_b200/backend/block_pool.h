// Host side of a paged cache: which block of the pool holds which page of which sequence. Blocks are handed out in
// arrival order, so the pages of the sequences that run together interleave in the pool, and the block freed last is
// the first to be used again.
#pragma once

#include <cstdint>
#include <stdexcept>
#include <vector>

class BlockPool {
public:
    BlockPool() = default;
    BlockPool(int n_blocks, int max_seqs, int pages_per_seq) : pages_per_seq_(pages_per_seq), table_(size_t(max_seqs) * size_t(pages_per_seq), -1) {
        for (int b = n_blocks - 1; b >= 0; b--) free_.push_back(b);
    }
    // Gives every page first..last of a sequence a block; pages that have one keep it.
    void ensure(int seq, int first, int last) {
        if (last >= pages_per_seq_) throw std::runtime_error("context window exceeded");
        int32_t* r = row(seq);
        for (int p = first; p <= last; p++) {
            if (r[p] >= 0) continue;
            if (free_.empty()) throw std::runtime_error("context window exceeded");
            r[p] = free_.back();
            free_.pop_back();
        }
    }
    // Gives back the blocks of pages first..last-1.
    void release(int seq, int first, int last) {
        int32_t* r = row(seq);
        for (int p = first; p < last; p++)
            if (r[p] >= 0) { free_.push_back(r[p]); r[p] = -1; }
    }
    void release(int seq) { release(seq, 0, pages_per_seq_); }
    int32_t* row(int seq) { return table_.data() + size_t(seq) * size_t(pages_per_seq_); }
    int pages_per_seq() const { return pages_per_seq_; }
    int free_blocks() const { return int(free_.size()); }

private:
    int pages_per_seq_ = 0;
    std::vector<int32_t> table_;  // [max_seqs][pages_per_seq], -1 = no block
    std::vector<int32_t> free_;
};
