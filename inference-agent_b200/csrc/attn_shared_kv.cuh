// Shared by the kernels of the shared-row attention (attn_shared_kv.cu, attn_shared_kv_sm100.cu): the cache handle, the
// page arithmetic and the launch parameters.
#pragma once

#include <cuda_bf16.h>

#include "attn_common.cuh"
#include "ingot_internal.cuh"

struct ingot_skv {
    int device = 0, num_sms = 0;
    int n_layer = 0, n_head_kv = 0, dim = 0;  // dim: row length (padded head size)
    int dtype = INGOT_F32, chunk = 0, window = 0, n_blocks = 0;
    bool tiled = false;  // pages in the order of page_elem()
    size_t layer_elems = 0;
    void* rows = nullptr;
    float* inv_rms = nullptr;  // [layer][block][16]; null in caches whose rows are the keys as they are (window form)
    int* status_dev = nullptr;
    float* part = nullptr;  // split-key partials of decoded tokens, grown on demand
    size_t part_floats = 0;
    std::vector<void*> retired;
    std::vector<CUtensorMap> tmaps;  // per layer, f16 rows in plain order: [page * kv head][16][row] in boxes of 16 x 64
};

// Which keys a position sees and which page holds it: the whole past, its own chunk, or a window that slides along.
struct PageMap {
    int chunk, pages_per_chunk;  // chunk 0: one chunk of unlimited length
    int window = 0;              // > 0 (chunk is 0 then): position i sees i - window + 1 .. i
    __host__ __device__ __forceinline__ int page(int pos) const { return chunk > 0 ? (pos / chunk) * pages_per_chunk + (pos % chunk) / kBlockTokens : pos / kBlockTokens; }
    __host__ __device__ __forceinline__ int slot(int pos) const { return (chunk > 0 ? pos % chunk : pos) % kBlockTokens; }
    __host__ __device__ __forceinline__ int first_visible(int pos) const {
        if (chunk > 0) return pos / chunk * chunk;
        return window > 0 && pos >= window ? pos - window + 1 : 0;
    }
};
inline PageMap page_map(const ingot_skv* kv) { return PageMap{kv->chunk, (kv->chunk + kBlockTokens - 1) / kBlockTokens, kv->window}; }

// Element of a page of one KV head that holds column `col` of slot `slot`. Plain: row after row. Tiled (f16 rows of whole 64-column
// units): [8-slot half][unit][8 slots][64 columns] with the 16-byte pieces of a slot XOR-swizzled by it - the shared-memory image the
// tcgen05 kernels multiply, so that a page comes in as one contiguous copy; the 8 values of a piece stay together.
__host__ __device__ __forceinline__ int page_elem(bool tiled, int row, int slot, int col) {
    if (!tiled) return slot * row + col;
    return (((slot >> 3) * (row >> 6) + (col >> 6)) * 8 + (slot & 7)) * 64 + ((((col >> 3) & 7) ^ (slot & 7)) << 3) + (col & 7);
}

struct SharedOut {
    float* f32;
    __nv_bfloat16 *hi, *lo;
    int ld;
    float scale;
    __device__ __forceinline__ void store(size_t row, int c, float v) const {
        const size_t i = row * ld + c;
        if (f32) f32[i] = v * scale;
        if (hi) {
            const __nv_bfloat16 h = __float2bfloat16_rn(v * scale);
            hi[i] = h;
            if (lo) lo[i] = __float2bfloat16_rn(v * scale - __bfloat162float(h));
        }
    }
    // Two neighbouring columns, c and ld even.
    __device__ __forceinline__ void store2(size_t row, int c, float a, float b) const {
        const size_t i = row * ld + c;
        a *= scale;
        b *= scale;
        if (f32) *reinterpret_cast<float2*>(f32 + i) = make_float2(a, b);
        if (hi) {
            const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
            *reinterpret_cast<__nv_bfloat162*>(hi + i) = h;
            if (lo) *reinterpret_cast<__nv_bfloat162*>(lo + i) = __floats2bfloat162_rn(a - __low2float(h), b - __high2float(h));
        }
    }
};

// A factor sigmoid(z) of the result: z one number per (token, head) or one per value (null: none).
struct OutGate {
    const float* z = nullptr;
    int ld = 0, per_head = 0;
    __device__ __forceinline__ static float sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
    __device__ __forceinline__ float at(size_t row, int head, int out_dim, int d) const {
        if (!z) return 1.0f;
        return sigmoid(z[row * ld + (per_head ? head : head * out_dim + d)]);
    }
};

// Block of a page of sequence `seq` (index within the step), or -1 with the status bit raised if the table has none.
__device__ __forceinline__ int table_block(const int32_t* tables, const int32_t* first_page, int max_blocks, int n_blocks, int seq, int page, int* status) {
    const int i = page - (first_page ? first_page[seq] : 0);
    const int blk = i >= 0 && i < max_blocks ? tables[(size_t)seq * max_blocks + i] : -1;
    if (blk >= 0 && blk < n_blocks) return blk;
    atomicOr(status, kDevErrBlockRange);
    return -1;
}

struct AttendParams {
    ingot_step st;
    const void* q;
    const void* rows;
    const float* inv_rms;  // null: keys have no scale of their own
    const int32_t *tables, *first_page;
    int max_blocks, n_blocks, n_head, n_head_kv, dim, out_dim;
    PageMap map;
    float scale;  // of the scores
    SharedOut out;
    int* status;
    int n_splits;   // decoding: CTAs per (token, KV head) over the keys
    float* part;    // [token][head][split][dim + 2]
    bool tiled = false;           // order of the pages
    const float* sink = nullptr;  // per head: one more term exp(sink) of the denominator (null: none)
    int q_dim = 0;                // columns of the row that are the key (0: all of them), and the first one of the value
    int v_off = 0;
    OutGate gate = {};
};

// The plain kernel (f32 arithmetic, any row length up to 1024, window, chunk and sink); dtype of rows and queries.
int launch_shared_kv_plain(const AttendParams& p, int dtype, cudaStream_t stream);

// Latent attention of decoded tokens on tcgen05 (attn_latent_decode_sm100.cu): which rows it takes, heads per CTA, and the launch for
// a step of single tokens (p.n_splits and p.part set).
bool latent_decode_takes(int row, int rank);
int latent_decode_heads(int n_head);
int launch_latent_decode_sm100(const ingot_skv* kv, const AttendParams& p, cudaStream_t stream);

// Attention over joined [key | value] rows for portions of prompts on tcgen05 (attn_gqa_sm100.cu): which sizes it takes, and the launch.
bool gqa_sm100_takes(int dim, int vdim, float scale);
int launch_gqa_sm100(ingot_skv* kv, int layer, const AttendParams& p, cudaStream_t stream);

// tcgen05 form for portions of prompts over rows of 128 values (attn_shared_kv_sm100.cu); INGOT_ERR_UNSUPPORTED if the driver
// cannot encode its tensor map.
int launch_shared_kv_sm100(ingot_skv* kv, int layer, const AttendParams& p, cudaStream_t stream);
