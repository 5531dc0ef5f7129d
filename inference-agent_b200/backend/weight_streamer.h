// Host-to-device weight upload.
#pragma once

#include <cuda_runtime.h>

#include <algorithm>
#include <cstring>

#include "cuda_util.h"

// Streams weights from the memory-mapped model file to the device through a small ring of pinned staging buffers:
// the CPU copy of chunk i+1 out of the page cache (where the page faults and disk reads happen) overlaps the DMA
// of chunk i, and no call blocks on a pageable copy. The Metal backend wraps the mmap without copying
// (src/metal_backend.mm:213-246); a discrete GPU has to move the bytes once, so they move as a stream.
class WeightStreamer {
public:
    WeightStreamer() {
        cuda_check(cudaStreamCreateWithFlags(&stream_, cudaStreamNonBlocking), "cudaStreamCreate(load)");
        for (int i = 0; i < kBufs; i++) {
            cuda_check(cudaMallocHost(&buf_[i], kChunk), "cudaMallocHost(load staging)");
            cuda_check(cudaEventCreateWithFlags(&done_[i], cudaEventDisableTiming), "cudaEventCreate");
        }
    }
    ~WeightStreamer() {
        cudaStreamSynchronize(stream_);
        for (int i = 0; i < kBufs; i++) { cudaFreeHost(buf_[i]); cudaEventDestroy(done_[i]); }
        cudaStreamDestroy(stream_);
    }
    void copy(void* dst_dev, const void* src_host, size_t bytes) {
        const char* src = static_cast<const char*>(src_host);
        char* dst = static_cast<char*>(dst_dev);
        for (size_t off = 0; off < bytes; off += kChunk) {
            const size_t n = std::min(kChunk, bytes - off);
            const int b = next_++ % kBufs;
            cuda_check(cudaEventSynchronize(done_[b]), "load staging");  // the DMA that last read this buffer is over
            memcpy(buf_[b], src + off, n);
            cuda_check(cudaMemcpyAsync(dst + off, buf_[b], n, cudaMemcpyHostToDevice, stream_), "cudaMemcpyAsync(weight)");
            cuda_check(cudaEventRecord(done_[b], stream_), "cudaEventRecord");
            bytes_ += n;
        }
    }
    cudaStream_t stream() const { return stream_; }
    void finish() { cuda_check(cudaStreamSynchronize(stream_), "weight upload"); }
    size_t bytes() const { return bytes_; }

private:
    static constexpr int kBufs = 4;
    static constexpr size_t kChunk = size_t(32) << 20;
    cudaStream_t stream_ = nullptr;
    void* buf_[kBufs] = {};
    cudaEvent_t done_[kBufs] = {};
    unsigned next_ = 0;
    size_t bytes_ = 0;
};
