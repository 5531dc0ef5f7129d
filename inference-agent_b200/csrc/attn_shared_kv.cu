// Attention over shared key/value rows: one cached row per token and KV head serves both as the key and as the value.
// No counterpart in the reference (its layers keep K and V apart, use RoPE and see the whole past).
//
// The mechanism. k = W_k h; the value of a token is k itself, the key is k normalised over the whole projection:
//     key = k / rms * w_k,  rms = sqrt(mean over all KV heads of k^2 + eps)
// so a cache row is k (not normalised) plus ONE f32 number 1/rms per token and layer: w_k goes into the query, and
//     score(i, j) = (q_i/rms_i * w_q * w_k) . k_j  * (1/rms_j) * scale.
// The cache and its traffic are half of a K + V cache. Positions do not enter the scores.
//
// Visibility: causal, and with chunk > 0 only inside the query's own chunk of `chunk` positions counted from position 0.
//
// Pages. A page is 16 consecutive positions of ONE chunk: page index of position p = (p / chunk) * ceil(chunk / 16) +
// (p % chunk) / 16 (chunk 0: p / 16), so a chunk begins on a page of its own and the pages of past chunks hold nothing
// that can be seen again - the owner of the block table may give them back. Layout [page][kv head][16][dim], f32 or f16,
// and [page][16] f32 for 1/rms.
#include <algorithm>
#include <new>

#include "ingot_internal.cuh"

#include <cuda_bf16.h>

struct ingot_skv {
    int device = 0, num_sms = 0;
    int n_layer = 0, n_head_kv = 0, dim = 0;  // dim: row length (padded head size)
    int dtype = INGOT_F32, chunk = 0, n_blocks = 0;
    size_t layer_elems = 0;
    void* rows = nullptr;
    float* inv_rms = nullptr;  // [layer][block][16]
    int* status_dev = nullptr;
};

namespace {

struct PageMap {
    int chunk, pages_per_chunk;  // chunk 0: one chunk of unlimited length
    __host__ __device__ __forceinline__ int page(int pos) const { return chunk > 0 ? (pos / chunk) * pages_per_chunk + (pos % chunk) / kBlockTokens : pos / kBlockTokens; }
    __host__ __device__ __forceinline__ int slot(int pos) const { return (chunk > 0 ? pos % chunk : pos) % kBlockTokens; }
    __host__ __device__ __forceinline__ int first_visible(int pos) const { return chunk > 0 ? pos / chunk * chunk : 0; }
};

struct SharedOut {
    float* f32;
    __nv_bfloat16* hi;
    int ld;
    float scale;
    __device__ __forceinline__ void store(size_t row, int c, float v) const {
        const size_t i = row * ld + c;
        if (f32) f32[i] = v * scale;
        if (hi) hi[i] = __float2bfloat16_rn(v * scale);
    }
};

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}
__device__ __forceinline__ float widen(float v) { return v; }
__device__ __forceinline__ float widen(__half v) { return __half2float(v); }
__device__ __forceinline__ void narrow(float* p, float v) { *p = v; }
__device__ __forceinline__ void narrow(__half* p, float v) { *p = __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f)); }

// One CTA per token: RMS of q and k over their whole projections, the folded query (rows [token][head][dim]), and the
// token's cache rows. q_cols / k_cols are n_head * dim and n_head_kv * dim columns of the projection row; the padding
// columns of a head are zero, so only the divisor of the mean (q_mean, k_mean: the unpadded counts) differs.
struct AppendParams {
    ingot_step st;
    const float* proj;
    int proj_ld, q_off, k_off, n_head, n_head_kv, dim, q_mean, k_mean;
    const float *wq, *wk;
    float eps;
    void* q_out;
    void* rows;
    float* inv_rms;
    const int32_t *tables, *first_page;
    int max_blocks, n_blocks;
    PageMap map;
    int* status;
};
// Block of a page of sequence `seq` (index within the step), or -1 with the status bit raised if the table has none.
__device__ __forceinline__ int table_block(const int32_t* tables, const int32_t* first_page, int max_blocks, int n_blocks, int seq, int page, int* status) {
    const int i = page - (first_page ? first_page[seq] : 0);
    const int blk = i >= 0 && i < max_blocks ? tables[(size_t)seq * max_blocks + i] : -1;
    if (blk >= 0 && blk < n_blocks) return blk;
    atomicOr(status, kDevErrBlockRange);
    return -1;
}
template <typename T>
__global__ void __launch_bounds__(128) shared_kv_append_kernel(const AppendParams p) {
    INGOT_PDL_TRIGGER();
    INGOT_PDL_WAIT();
    __shared__ float red[8];
    const int row = blockIdx.x, seq = p.st.row_seq[row];
    const int pos = p.st.pos0[seq] + row - p.st.row_start[seq];
    const float* q = p.proj + (size_t)row * p.proj_ld + p.q_off;
    const float* k = p.proj + (size_t)row * p.proj_ld + p.k_off;
    const int nq = p.n_head * p.dim, nk = p.n_head_kv * p.dim;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < nq; i += 128) sq = fmaf(q[i], q[i], sq);
    for (int i = threadIdx.x; i < nk; i += 128) sk = fmaf(k[i], k[i], sk);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) { red[threadIdx.x >> 5] = sq; red[4 + (threadIdx.x >> 5)] = sk; }
    __syncthreads();
    const float iq = 1.0f / sqrtf((red[0] + red[1] + red[2] + red[3]) / float(p.q_mean) + p.eps);
    const float ik = 1.0f / sqrtf((red[4] + red[5] + red[6] + red[7]) / float(p.k_mean) + p.eps);
    T* qo = static_cast<T*>(p.q_out) + (size_t)row * nq;
    const int group = p.n_head / p.n_head_kv;
    for (int i = threadIdx.x; i < nq; i += 128) {
        const int h = i / p.dim, d = i - h * p.dim;
        narrow(qo + i, q[i] * iq * p.wq[i] * p.wk[(h / group) * p.dim + d]);
    }
    const int page = p.map.page(pos), slot = p.map.slot(pos);
    const int blk = table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, page, p.status);
    if (blk < 0) return;
    for (int i = threadIdx.x; i < nk; i += 128) {
        const int h = i / p.dim, d = i - h * p.dim;
        narrow(static_cast<T*>(p.rows) + (((size_t)blk * p.n_head_kv + h) * kBlockTokens + slot) * p.dim + d, k[i]);
    }
    if (threadIdx.x == 0) p.inv_rms[(size_t)blk * kBlockTokens + slot] = ik;
}

struct AttendParams {
    ingot_step st;
    const void* q;
    const void* rows;
    const float* inv_rms;
    const int32_t *tables, *first_page;
    int max_blocks, n_blocks, n_head, n_head_kv, dim, out_dim;
    PageMap map;
    float scale;
    SharedOut out;
    int* status;
};

// ---- plain form: f32 arithmetic on the FMA pipes, any row length up to 512, f32 or f16 rows -------------------------
// A CTA owns 16 (token, head) rows of one KV head - 4 per warp - and walks the visible keys 32 at a time through shared
// memory: lane = key for the scores, lane = dims for the weighted sum.
constexpr int kRows = 16, kKeys = 32;
template <typename T, int kD>  // kD: row length in units of 32, rounded up
__global__ void __launch_bounds__(128) shared_kv_attend_kernel(const AttendParams p) {
    extern __shared__ __align__(16) float smem[];
    INGOT_PDL_TRIGGER();
    INGOT_PDL_WAIT();
    const int seq = blockIdx.z, kvh = blockIdx.y;
    const int group = p.n_head / p.n_head_kv, len = p.st.len[seq];
    const int row0 = blockIdx.x * kRows, n_rows = len * group;
    if (row0 >= n_rows) return;
    const int dim = p.dim, ldk = kD * 32 + 1;
    float* sq = smem;                       // [16][kD * 32]
    float* sk = sq + kRows * kD * 32;       // [32][kD * 32 + 1]
    float* sr = sk + kKeys * ldk;           // [32] 1/rms * scale
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos0 = p.st.pos0[seq];
    const size_t tok0 = p.st.row_start[seq];

    for (int i = threadIdx.x; i < kRows * kD * 32; i += 128) {
        const int r = i / (kD * 32), d = i - r * (kD * 32);
        const int rr = row0 + r;
        float v = 0.f;
        if (rr < n_rows && d < dim) v = widen(static_cast<const T*>(p.q)[((tok0 + rr / group) * p.n_head + kvh * group + rr % group) * dim + d]);
        sq[i] = v;
    }
    int lo[4], hi[4];  // visible keys lo..hi of this warp's rows (none: hi < lo)
    float m[4], l[4], acc[4][kD];
#pragma unroll
    for (int r = 0; r < 4; r++) {
        const int rr = row0 + warp * 4 + r;
        const int pos = pos0 + rr / group;
        lo[r] = rr < n_rows ? p.map.first_visible(pos) : 0;
        hi[r] = rr < n_rows ? pos : -1;
        m[r] = -INFINITY;
        l[r] = 0.f;
#pragma unroll
        for (int i = 0; i < kD; i++) acc[r][i] = 0.f;
    }
    const int first = p.map.first_visible(pos0 + row0 / group);
    const int last = pos0 + (min(row0 + kRows, n_rows) - 1) / group;
    for (int j0 = first; j0 <= last; j0 += kKeys) {
        __syncthreads();
        {
            const int key = threadIdx.x >> 2, part = threadIdx.x & 3;
            const int j = j0 + key;
            int blk = -1, slot = 0;
            if (j <= last) {
                slot = p.map.slot(j);
                blk = table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, p.map.page(j), p.status);
            }
            const T* src = static_cast<const T*>(p.rows) + (((size_t)max(blk, 0) * p.n_head_kv + kvh) * kBlockTokens + slot) * dim;
            for (int d = part; d < kD * 32; d += 4) sk[key * ldk + d] = blk >= 0 && d < dim ? widen(src[d]) : 0.f;
            if (part == 0) sr[key] = blk >= 0 ? p.inv_rms[(size_t)blk * kBlockTokens + slot] * p.scale : 0.f;
        }
        __syncthreads();
        const int j = j0 + lane;
#pragma unroll
        for (int r = 0; r < 4; r++) {
            if (hi[r] < j0 || lo[r] >= j0 + kKeys) continue;  // warp-uniform
            const float* qr = sq + (warp * 4 + r) * kD * 32;
            const float* kr = sk + lane * ldk;
            float s0 = 0.f, s1 = 0.f;
            for (int d = 0; d < dim; d += 2) {
                s0 = fmaf(qr[d], kr[d], s0);
                s1 = fmaf(qr[d + 1], kr[d + 1], s1);
            }
            const bool on = j >= lo[r] && j <= hi[r];
            const float s = on ? (s0 + s1) * sr[lane] : -INFINITY;
            const float m_new = fmaxf(m[r], warp_max(s));
            const float alpha = expf(m[r] - m_new);
            const float e = on ? expf(s - m_new) : 0.f;
            l[r] = l[r] * alpha + warp_sum(e);
            m[r] = m_new;
#pragma unroll
            for (int i = 0; i < kD; i++) acc[r][i] *= alpha;
            for (int k = 0; k < kKeys; k++) {
                const float pk = __shfl_sync(0xffffffffu, e, k);
                if (pk == 0.f) continue;  // warp-uniform
#pragma unroll
                for (int i = 0; i < kD; i++) acc[r][i] = fmaf(pk, sk[k * ldk + lane + 32 * i], acc[r][i]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < 4; r++) {
        const int rr = row0 + warp * 4 + r;
        if (rr >= n_rows) continue;
        const float inv = 1.0f / l[r];
#pragma unroll
        for (int i = 0; i < kD; i++) {
            const int d = lane + 32 * i;
            if (d < p.out_dim) p.out.store(tok0 + rr / group, (kvh * group + rr % group) * p.out_dim + d, acc[r][i] * inv);
        }
    }
}

template <typename T>
int launch_plain(const AttendParams& p, cudaStream_t s) {
    const int group = p.n_head / p.n_head_kv;
    const dim3 grid((unsigned)(((size_t)p.st.max_len * group + kRows - 1) / kRows), p.n_head_kv, p.st.n_seq);
    const int units = (p.dim + 31) / 32;
    const int kd = units <= 1 ? 1 : units <= 2 ? 2 : units <= 4 ? 4 : units <= 8 ? 8 : 16;
    const size_t smem = ((size_t)kRows * kd * 32 + (size_t)kKeys * (kd * 32 + 1) + kKeys) * sizeof(float);
    auto kernel = kd == 1 ? shared_kv_attend_kernel<T, 1> : kd == 2 ? shared_kv_attend_kernel<T, 2> : kd == 4 ? shared_kv_attend_kernel<T, 4>
                : kd == 8 ? shared_kv_attend_kernel<T, 8> : shared_kv_attend_kernel<T, 16>;
    if (smem > 48 * 1024) INGOT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    INGOT_CUDA_TRY(ingot_launch_pdl(kernel, grid, dim3(128), smem, s, p));
    return INGOT_OK;
}

bool step_ok(const ingot_step* st) {
    return st && st->n_tok >= 1 && st->n_seq >= 1 && st->n_seq <= 65535 && st->max_len >= 1 && st->row_seq && st->row_start && st->len && st->pos0;
}

}  // namespace

extern "C" {

int ingot_skv_create(ingot_skv** out, int n_layer, int n_head_kv, int head_dim, int dtype, int chunk, int n_blocks) {
    INGOT_REQUIRE(out != nullptr, "ingot_skv_create: out is null");
    *out = nullptr;
    INGOT_REQUIRE(n_layer >= 1 && n_head_kv >= 1 && n_blocks >= 1 && chunk >= 0, "ingot_skv_create: bad sizes");
    INGOT_REQUIRE(dtype == INGOT_F32 || dtype == INGOT_F16, "ingot_skv_create: rows are f32 or f16");
    if (head_dim < 2 || head_dim > 512 || head_dim % 2 != 0) {
        ingot_set_error("ingot_skv_create: row length must be even and at most 512");
        return INGOT_ERR_UNSUPPORTED;
    }
    ingot_skv* kv = new (std::nothrow) ingot_skv();
    if (!kv) return INGOT_ERR_NOMEM;
    kv->n_layer = n_layer; kv->n_head_kv = n_head_kv; kv->dim = head_dim; kv->dtype = dtype; kv->chunk = chunk; kv->n_blocks = n_blocks;
    kv->layer_elems = (size_t)n_blocks * n_head_kv * kBlockTokens * head_dim;
    const size_t bytes = kv->layer_elems * n_layer * (dtype == INGOT_F32 ? 4 : 2), scale_bytes = (size_t)n_layer * n_blocks * kBlockTokens * 4;
    cudaError_t e;
    // zero-filled: rows that were never written stay finite, so a masked key cannot inject NaN through 0 * garbage
    if ((e = cudaGetDevice(&kv->device)) != cudaSuccess || (e = cudaDeviceGetAttribute(&kv->num_sms, cudaDevAttrMultiProcessorCount, kv->device)) != cudaSuccess ||
        (e = cudaMalloc(&kv->rows, bytes)) != cudaSuccess || (e = cudaMalloc(&kv->inv_rms, scale_bytes)) != cudaSuccess ||
        (e = cudaMalloc(&kv->status_dev, sizeof(int))) != cudaSuccess || (e = cudaMemset(kv->rows, 0, bytes)) != cudaSuccess ||
        (e = cudaMemset(kv->inv_rms, 0, scale_bytes)) != cudaSuccess || (e = cudaMemset(kv->status_dev, 0, sizeof(int))) != cudaSuccess ||
        (e = cudaDeviceSynchronize()) != cudaSuccess) {
        const int rc = ingot_cuda_fail(e, "ingot_skv_create");
        ingot_skv_destroy(kv);
        return rc;
    }
    *out = kv;
    return INGOT_OK;
}

void ingot_skv_destroy(ingot_skv* kv) {
    if (!kv) return;
    cudaFree(kv->rows);
    cudaFree(kv->inv_rms);
    cudaFree(kv->status_dev);
    delete kv;
}

int ingot_skv_pages(int chunk, int n_positions) {
    if (n_positions < 1 || chunk < 0) return 0;
    const PageMap map = {chunk, (chunk + kBlockTokens - 1) / kBlockTokens};
    return map.page(n_positions - 1) + 1;
}

int* ingot_skv_status_dev(ingot_skv* kv) { return kv ? kv->status_dev : nullptr; }

int ingot_skv_row_length(int head_size) { return head_size < 1 ? 0 : (head_size + 15) / 16 * 16; }

int ingot_skv_status(ingot_skv* kv, void* stream, int* status_out) {
    INGOT_REQUIRE(kv && status_out, "ingot_skv_status: null argument");
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    INGOT_CUDA_TRY(cudaMemcpyAsync(status_out, kv->status_dev, sizeof(int), cudaMemcpyDeviceToHost, s));
    INGOT_CUDA_TRY(cudaMemsetAsync(kv->status_dev, 0, sizeof(int), s));
    INGOT_CUDA_TRY(cudaStreamSynchronize(s));
    return INGOT_OK;
}

int ingot_skv_append(ingot_skv* kv, int layer, const ingot_step* step, const float* proj_dev, int proj_ld, int q_off, int k_off,
                     int n_head, int head_size, const float* q_norm_dev, const float* k_norm_dev, float eps, void* q_out_dev,
                     const int32_t* tables_dev, const int32_t* first_page_dev, int max_blocks, void* stream) {
    INGOT_REQUIRE(kv && step_ok(step), "ingot_skv_append: null handle or bad step");
    INGOT_REQUIRE_DEVICE(kv);
    INGOT_REQUIRE(layer >= 0 && layer < kv->n_layer, "ingot_skv_append: layer out of range");
    INGOT_REQUIRE(proj_dev && q_norm_dev && k_norm_dev && q_out_dev && tables_dev && max_blocks >= 1, "ingot_skv_append: null argument");
    INGOT_REQUIRE(n_head >= kv->n_head_kv && n_head % kv->n_head_kv == 0, "ingot_skv_append: n_head must be a multiple of n_head_kv");
    INGOT_REQUIRE(head_size >= 1 && head_size <= kv->dim, "ingot_skv_append: head size beyond the row length");
    const size_t esz = kv->dtype == INGOT_F32 ? 4 : 2;
    AppendParams p = {*step, proj_dev, proj_ld, q_off, k_off, n_head, kv->n_head_kv, kv->dim, n_head * head_size, kv->n_head_kv * head_size,
                      q_norm_dev, k_norm_dev, eps, q_out_dev, static_cast<char*>(kv->rows) + kv->layer_elems * layer * esz,
                      kv->inv_rms + (size_t)layer * kv->n_blocks * kBlockTokens, tables_dev, first_page_dev, max_blocks, kv->n_blocks,
                      PageMap{kv->chunk, (kv->chunk + kBlockTokens - 1) / kBlockTokens}, kv->status_dev};
    auto kernel = kv->dtype == INGOT_F32 ? shared_kv_append_kernel<float> : shared_kv_append_kernel<__half>;
    INGOT_CUDA_TRY(ingot_launch_pdl(kernel, dim3(step->n_tok), dim3(128), 0, static_cast<cudaStream_t>(stream), p));
    return INGOT_OK;
}

int ingot_skv_attend(ingot_skv* kv, int layer, const ingot_step* step, const void* q_dev, int n_head, int out_dim, float scale,
                     float out_scale, const ingot_act_out* out, const int32_t* tables_dev, const int32_t* first_page_dev, int max_blocks, int impl, void* stream) {
    INGOT_REQUIRE(kv && step_ok(step), "ingot_skv_attend: null handle or bad step");
    INGOT_REQUIRE_DEVICE(kv);
    INGOT_REQUIRE(layer >= 0 && layer < kv->n_layer, "ingot_skv_attend: layer out of range");
    INGOT_REQUIRE(q_dev && out && tables_dev && max_blocks >= 1, "ingot_skv_attend: null argument");
    INGOT_REQUIRE(n_head >= kv->n_head_kv && n_head % kv->n_head_kv == 0, "ingot_skv_attend: n_head must be a multiple of n_head_kv");
    INGOT_REQUIRE(out_dim >= 1 && out_dim <= kv->dim && !out->lo, "ingot_skv_attend: bad output");
    (void)impl;
    const size_t esz = kv->dtype == INGOT_F32 ? 4 : 2;
    AttendParams p = {*step, q_dev, static_cast<const char*>(kv->rows) + kv->layer_elems * layer * esz,
                      kv->inv_rms + (size_t)layer * kv->n_blocks * kBlockTokens, tables_dev, first_page_dev, max_blocks, kv->n_blocks, n_head, kv->n_head_kv,
                      kv->dim, out_dim, PageMap{kv->chunk, (kv->chunk + kBlockTokens - 1) / kBlockTokens}, scale,
                      SharedOut{out->f32, static_cast<__nv_bfloat16*>(out->hi), out->ld, out_scale}, kv->status_dev};
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    return kv->dtype == INGOT_F32 ? launch_plain<float>(p, s) : launch_plain<__half>(p, s);
}

}  // extern "C"
