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

#include "attn_shared_kv.cuh"

namespace {

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
__device__ __forceinline__ void narrow(__half* p, float v) { *p = __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f)); }

__device__ __forceinline__ void narrow4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void narrow4(__half* p, float4 v) {
    __half h[4];
    narrow(h, v.x); narrow(h + 1, v.y); narrow(h + 2, v.z); narrow(h + 3, v.w);
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(h);
}

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
constexpr int kAppendThreads = 256;
template <typename T>
__global__ void __launch_bounds__(kAppendThreads) shared_kv_append_kernel(const AppendParams p) {
    INGOT_PDL_TRIGGER();
    INGOT_PDL_WAIT();
    __shared__ float red[2 * kAppendThreads / 32];
    const int row = blockIdx.x, seq = p.st.row_seq[row];
    const int pos = p.st.pos0[seq] + row - p.st.row_start[seq];
    const float* q = p.proj + (size_t)row * p.proj_ld + p.q_off;
    const float* k = p.proj + (size_t)row * p.proj_ld + p.k_off;
    const int nq = p.n_head * p.dim, nk = p.n_head_kv * p.dim;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x * 4; i < nq; i += kAppendThreads * 4) {
        const float4 v = *reinterpret_cast<const float4*>(q + i);
        sq = fmaf(v.x, v.x, sq); sq = fmaf(v.y, v.y, sq); sq = fmaf(v.z, v.z, sq); sq = fmaf(v.w, v.w, sq);
    }
    for (int i = threadIdx.x * 4; i < nk; i += kAppendThreads * 4) {
        const float4 v = *reinterpret_cast<const float4*>(k + i);
        sk = fmaf(v.x, v.x, sk); sk = fmaf(v.y, v.y, sk); sk = fmaf(v.z, v.z, sk); sk = fmaf(v.w, v.w, sk);
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (lane == 0) { red[warp] = sq; red[kAppendThreads / 32 + warp] = sk; }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < kAppendThreads / 32; w++) { sq += red[w]; sk += red[kAppendThreads / 32 + w]; }
    const float iq = 1.0f / sqrtf(sq / float(p.q_mean) + p.eps);
    const float ik = 1.0f / sqrtf(sk / float(p.k_mean) + p.eps);
    T* qo = static_cast<T*>(p.q_out) + (size_t)row * nq;
    const int group = p.n_head / p.n_head_kv;
    for (int h = warp; h < p.n_head; h += kAppendThreads / 32) {
        const float* wk = p.wk + (h / group) * p.dim;
        for (int d = lane * 4; d < p.dim; d += 128) {
            const int i = h * p.dim + d;
            const float4 v = *reinterpret_cast<const float4*>(q + i), a = *reinterpret_cast<const float4*>(p.wq + i), b = *reinterpret_cast<const float4*>(wk + d);
            narrow4(qo + i, make_float4(v.x * iq * a.x * b.x, v.y * iq * a.y * b.y, v.z * iq * a.z * b.z, v.w * iq * a.w * b.w));
        }
    }
    const int page = p.map.page(pos), slot = p.map.slot(pos);
    const int blk = table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, page, p.status);
    if (blk < 0) return;
    for (int h = warp; h < p.n_head_kv; h += kAppendThreads / 32) {
        T* dst = static_cast<T*>(p.rows) + (((size_t)blk * p.n_head_kv + h) * kBlockTokens + slot) * p.dim;
        for (int d = lane * 4; d < p.dim; d += 128) narrow4(dst + d, *reinterpret_cast<const float4*>(k + h * p.dim + d));
    }
    if (threadIdx.x == 0) p.inv_rms[(size_t)blk * kBlockTokens + slot] = ik;
}

// ---- plain form: f32 arithmetic on the FMA pipes, any row length up to 1024, f32 or f16 rows -------------------------
// The key is the row or its first q_dim columns, the value its out_dim columns from v_off on.
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
    const int dim = p.dim, ldk = kD * 32 + 1, q_dim = p.q_dim > 0 ? p.q_dim : dim;
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
        if (rr < n_rows && d < q_dim) v = widen(static_cast<const T*>(p.q)[((tok0 + rr / group) * p.n_head + kvh * group + rr % group) * q_dim + d]);
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
            const T* src = static_cast<const T*>(p.rows) + ((size_t)max(blk, 0) * p.n_head_kv + kvh) * kBlockTokens * dim;
            for (int d = part; d < kD * 32; d += 4) sk[key * ldk + d] = blk >= 0 && d < dim ? widen(src[page_elem(p.tiled, dim, slot, d)]) : 0.f;
            if (part == 0) sr[key] = blk < 0 ? 0.f : p.inv_rms ? p.inv_rms[(size_t)blk * kBlockTokens + slot] * p.scale : p.scale;
        }
        __syncthreads();
        const int j = j0 + lane;
#pragma unroll
        for (int r = 0; r < 4; r++) {
            if (hi[r] < j0 || lo[r] >= j0 + kKeys) continue;  // warp-uniform
            const float* qr = sq + (warp * 4 + r) * kD * 32;
            const float* kr = sk + lane * ldk;
            float s0 = 0.f, s1 = 0.f;
            for (int d = 0; d < q_dim; d += 2) {
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
                for (int i = 0; i < kD; i++)
                    if (p.v_off + 32 * i < kD * 32) acc[r][i] = fmaf(pk, sk[k * ldk + p.v_off + lane + 32 * i], acc[r][i]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < 4; r++) {
        const int rr = row0 + warp * 4 + r;
        if (rr >= n_rows) continue;
        float inv = 1.0f / l[r];
        if (p.sink) {
            const float sink = p.sink[kvh * group + rr % group], top = fmaxf(m[r], sink), mine = expf(m[r] - top);
            inv = mine / (l[r] * mine + expf(sink - top));
        }
#pragma unroll
        for (int i = 0; i < kD; i++) {
            const int d = lane + 32 * i;
            const size_t row = tok0 + rr / group;
            const int h = kvh * group + rr % group;
            if (d < p.out_dim) p.out.store(row, h * p.out_dim + d, acc[r][i] * inv * p.gate.at(row, h, p.out_dim, d));
        }
    }
}

template <typename T>
int launch_plain(const AttendParams& p, cudaStream_t s) {
    const int group = p.n_head / p.n_head_kv;
    const dim3 grid((unsigned)(((size_t)p.st.max_len * group + kRows - 1) / kRows), p.n_head_kv, p.st.n_seq);
    const int units = (p.dim + 31) / 32;
    const int kd = units <= 1 ? 1 : units <= 2 ? 2 : units <= 4 ? 4 : units <= 8 ? 8 : units <= 16 ? 16 : units <= 20 ? 20 : 32;
    const size_t smem = ((size_t)kRows * kd * 32 + (size_t)kKeys * (kd * 32 + 1) + kKeys) * sizeof(float);
    auto kernel = kd == 1 ? shared_kv_attend_kernel<T, 1> : kd == 2 ? shared_kv_attend_kernel<T, 2> : kd == 4 ? shared_kv_attend_kernel<T, 4>
                : kd == 8 ? shared_kv_attend_kernel<T, 8> : kd == 16 ? shared_kv_attend_kernel<T, 16> : kd == 20 ? shared_kv_attend_kernel<T, 20>
                : shared_kv_attend_kernel<T, 32>;
    if (smem > 48 * 1024) INGOT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    INGOT_CUDA_TRY(ingot_launch_pdl(kernel, grid, dim3(128), smem, s, p));
    return INGOT_OK;
}

// ---- tensor-core form: f16 rows, m16n8k16 MMAs, one shared-memory tile for both products ------------------------------
// Because a cached row is key and value at once, a staged tile serves S = Q K^T (plain ldmatrix) and O += P V (transposing
// ldmatrix): half the copies and half the shared memory of a K + V kernel. Tiles are 64 keys = 4 pages, fetched page by page
// with cp.async; the key's scale (1/rms * score scale) and its position travel with the tile, and the scale multiplies the
// f32 score.
// 8 warps of 16 (token, head) rows each share every tile.
constexpr int kTileKeys = 64;
constexpr int kSplitKeysMin = 128;
template <int kDim> struct MmaTile {
    static constexpr int kStride = kDim + 8;  // halves; rows start 4 banks apart (mod 32 a permutation), so ldmatrix is conflict-free
    static constexpr int kBytes = kTileKeys * kStride * 2;
};
__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool on) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(on ? 16 : 0) : "memory");
}

template <int kDim>
__global__ void __launch_bounds__(256) shared_kv_mma_kernel(const AttendParams p) {
    constexpr int kThreads = 256, kWarps = kThreads / 32, kStages = 2;
    constexpr int kStride = MmaTile<kDim>::kStride, kK = kDim / 16, kNt = kTileKeys / 8;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    INGOT_PDL_TRIGGER();
    INGOT_PDL_WAIT();
    const int seq = blockIdx.z, group = p.n_head / p.n_head_kv;
    const int kvh = blockIdx.y, len = p.st.len[seq], n_rows = len * group;
    // prompts: later tiles see more keys, they go first
    constexpr int tile_rows = kWarps * 16;
    const int row0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * tile_rows;
    if (row0 >= n_rows) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j = lane & 3;
    const int pos0 = p.st.pos0[seq];
    const size_t tok0 = p.st.row_start[seq];
    const __half* rows = static_cast<const __half*>(p.rows);

    const int pos_first = pos0 + row0 / group, pos_last = pos0 + (min(row0 + tile_rows, n_rows) - 1) / group;
    const int page_a = p.map.page(p.map.first_visible(pos_first)), page_b = p.map.page(pos_last);
    const int n_tiles = (page_b - page_a) / 4 + 1;

    // this thread's two rows
    const int r_lo = row0 + warp * 16 + g, r_hi = r_lo + 8;
    const int pos_lo = pos0 + min(r_lo, n_rows - 1) / group, pos_hi = pos0 + min(r_hi, n_rows - 1) / group;
    const int vis_lo = p.map.first_visible(pos_lo), vis_hi = p.map.first_visible(pos_hi);
    uint32_t qf[kK][4];
    {
        const __half* q = static_cast<const __half*>(p.q);
        const __half* a = q + ((tok0 + r_lo / group) * p.n_head + kvh * group + r_lo % group) * kDim;
        const __half* b = q + ((tok0 + r_hi / group) * p.n_head + kvh * group + r_hi % group) * kDim;
#pragma unroll
        for (int k = 0; k < kK; k++) {
            qf[k][0] = r_lo < n_rows ? *reinterpret_cast<const uint32_t*>(a + k * 16 + 2 * j) : 0u;
            qf[k][1] = r_hi < n_rows ? *reinterpret_cast<const uint32_t*>(b + k * 16 + 2 * j) : 0u;
            qf[k][2] = r_lo < n_rows ? *reinterpret_cast<const uint32_t*>(a + k * 16 + 8 + 2 * j) : 0u;
            qf[k][3] = r_hi < n_rows ? *reinterpret_cast<const uint32_t*>(b + k * 16 + 8 + 2 * j) : 0u;
        }
    }

    const uint32_t s_tile = (uint32_t)__cvta_generic_to_shared(smem_raw);
    float* s_scale = reinterpret_cast<float*>(smem_raw + kStages * MmaTile<kDim>::kBytes);  // [stage][64]
    int* s_pos = reinterpret_cast<int*>(s_scale + kStages * kTileKeys);                      // [stage][64]: position, or INT_MAX

    auto stage = [&](int t, int buf) {
        constexpr int kPieces = kDim / 8;
        for (int i = threadIdx.x; i < kTileKeys * kPieces; i += kThreads) {
            const int key = i / kPieces, c = i - key * kPieces;
            const int page = page_a + t * 4 + (key >> 4);
            const int blk = page <= page_b ? table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, page, p.status) : -1;
            const __half* src = rows + (((size_t)max(blk, 0) * p.n_head_kv + kvh) * kBlockTokens + (key & 15)) * kDim + c * 8;
            cp16(s_tile + buf * MmaTile<kDim>::kBytes + (key * kStride + c * 8) * 2, src, blk >= 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (threadIdx.x < kTileKeys) {
            const int key = threadIdx.x, page = page_a + t * 4 + (key >> 4);
            const int blk = page <= page_b ? table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, page, p.status) : -1;
            int pos = 0x7fffffff;
            if (blk >= 0) {
                if (p.map.chunk > 0) {
                    const int c = page / p.map.pages_per_chunk, rel = (page - c * p.map.pages_per_chunk) * kBlockTokens + (key & 15);
                    if (rel < p.map.chunk) pos = c * p.map.chunk + rel;
                } else {
                    pos = page * kBlockTokens + (key & 15);
                }
            }
            s_pos[buf * kTileKeys + key] = pos;
            s_scale[buf * kTileKeys + key] = blk >= 0 ? p.inv_rms[(size_t)blk * kBlockTokens + (key & 15)] * p.scale * 1.44269504f : 0.f;
        }
    };

    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    float o[kDim / 8][4];
#pragma unroll
    for (int i = 0; i < kDim / 8; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;

#pragma unroll
    for (int i = 0; i < kStages - 1; i++) {
        if (i < n_tiles) stage(i, i);
        else asm volatile("cp.async.commit_group;" ::: "memory");
    }
    for (int t = 0; t < n_tiles; t++) {
        const int buf = t % kStages;
        asm volatile("cp.async.wait_group %0;" ::"n"(kStages - 2) : "memory");
        __syncthreads();  // tile t is in, and every warp is done with the buffer that is staged next
        if (t + kStages - 1 < n_tiles) stage(t + kStages - 1, (t + kStages - 1) % kStages);
        else asm volatile("cp.async.commit_group;" ::: "memory");
        const uint32_t tile = s_tile + buf * MmaTile<kDim>::kBytes;
        const float* sc = s_scale + buf * kTileKeys;
        const int* kp = s_pos + buf * kTileKeys;

        float s[kNt][4];
#pragma unroll
        for (int nt = 0; nt < kNt; nt += 2) {
#pragma unroll
            for (int e = 0; e < 4; e++) s[nt][e] = s[nt + 1][e] = 0.f;
            // matrices: keys nt*8.. dims 0-7, same keys dims 8-15, keys (nt+1)*8.. dims 0-7, dims 8-15
            const uint32_t a = tile + ((nt * 8 + (lane & 7) + ((lane >> 4) & 1) * 8) * kStride + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
            for (int k = 0; k < kK; k++) {
                uint32_t b[4];
                ldmatrix4(b, a + k * 32);
                mma_16816(s[nt], qf[k][0], qf[k][1], qf[k][2], qf[k][3], b[0], b[1]);
                mma_16816(s[nt + 1], qf[k][0], qf[k][1], qf[k][2], qf[k][3], b[2], b[3]);
            }
        }
        // scale and mask; a tile all of whose keys every row of the CTA sees needs no mask
        const bool masked = s_pos[buf * kTileKeys] < p.map.first_visible(pos_last) || s_pos[buf * kTileKeys + kTileKeys - 1] > pos_first ||
                            (p.map.chunk > 0 && p.map.chunk % kBlockTokens != 0);
        float mx_lo = -INFINITY, mx_hi = -INFINITY;
#pragma unroll
        for (int nt = 0; nt < kNt; nt++) {
            const float2 ks = *reinterpret_cast<const float2*>(sc + nt * 8 + 2 * j);
            s[nt][0] *= ks.x; s[nt][1] *= ks.y; s[nt][2] *= ks.x; s[nt][3] *= ks.y;
            if (masked) {
                const int2 kpos = *reinterpret_cast<const int2*>(kp + nt * 8 + 2 * j);
                if (kpos.x < vis_lo || kpos.x > pos_lo) s[nt][0] = -INFINITY;
                if (kpos.y < vis_lo || kpos.y > pos_lo) s[nt][1] = -INFINITY;
                if (kpos.x < vis_hi || kpos.x > pos_hi) s[nt][2] = -INFINITY;
                if (kpos.y < vis_hi || kpos.y > pos_hi) s[nt][3] = -INFINITY;
            }
            mx_lo = fmaxf(mx_lo, fmaxf(s[nt][0], s[nt][1]));
            mx_hi = fmaxf(mx_hi, fmaxf(s[nt][2], s[nt][3]));
        }
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
        const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);
        // a row that has not seen a key yet keeps -inf; 0 stands in for it in the exponents
        const float rf_lo = mn_lo == -INFINITY ? 0.f : mn_lo, rf_hi = mn_hi == -INFINITY ? 0.f : mn_hi;
        const float a_lo = exp2f(m_lo - rf_lo), a_hi = exp2f(m_hi - rf_hi);
        m_lo = mn_lo;
        m_hi = mn_hi;
        float sum_lo = 0.f, sum_hi = 0.f;
        uint32_t pa[kNt][2];
#pragma unroll
        for (int nt = 0; nt < kNt; nt++) {
            const float p0 = exp2f(s[nt][0] - rf_lo), p1 = exp2f(s[nt][1] - rf_lo), p2 = exp2f(s[nt][2] - rf_hi), p3 = exp2f(s[nt][3] - rf_hi);
            sum_lo += p0 + p1;
            sum_hi += p2 + p3;
            pa[nt][0] = pack_half2_rn(p0, p1);
            pa[nt][1] = pack_half2_rn(p2, p3);
        }
        l_lo = l_lo * a_lo + sum_lo;
        l_hi = l_hi * a_hi + sum_hi;
        if (a_lo != 1.f || a_hi != 1.f) {
#pragma unroll
            for (int i = 0; i < kDim / 8; i++) { o[i][0] *= a_lo; o[i][1] *= a_lo; o[i][2] *= a_hi; o[i][3] *= a_hi; }
        }
        // O += P V; transposed 8x8 matrices: keys 0-7 dims d.., keys 8-15 dims d.., keys 0-7 dims d+8.., keys 8-15 dims d+8..
#pragma unroll
        for (int kk = 0; kk < kNt / 2; kk++) {
            const uint32_t a = tile + ((kk * 16 + (lane & 15)) * kStride + (lane >> 4) * 8) * 2;
#pragma unroll
            for (int d = 0; d < kDim / 16; d++) {
                uint32_t b[4];
                ldmatrix4_trans(b, a + d * 32);
                mma_16816(o[2 * d], pa[2 * kk][0], pa[2 * kk][1], pa[2 * kk + 1][0], pa[2 * kk + 1][1], b[0], b[1]);
                mma_16816(o[2 * d + 1], pa[2 * kk][0], pa[2 * kk][1], pa[2 * kk + 1][0], pa[2 * kk + 1][1], b[2], b[3]);
            }
        }
    }
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);

    const float i_lo = 1.0f / l_lo, i_hi = 1.0f / l_hi;
#pragma unroll
    for (int half = 0; half < 2; half++) {
        const int r = half ? r_hi : r_lo;
        if (r >= n_rows) continue;
        const size_t row = tok0 + r / group;
        const int c0 = (kvh * group + r % group) * p.out_dim;
        const float inv = half ? i_hi : i_lo;
#pragma unroll
        for (int i = 0; i < kDim / 8; i++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int d = i * 8 + 2 * j + e;
                if (d < p.out_dim) p.out.store(row, c0 + d, o[i][half * 2 + e] * inv);
            }
    }
}

// ---- decoding: one token of a sequence, split keys -------------------------------------------------------------------
// A CTA serves the heads of one token that read one KV head (16 rows of the MMAs) over one share of the visible pages. Its four
// warps take every fourth page each, through a cp.async ring of their own - no barrier in the key loop - with the page's 1/rms
// travelling along; the block table of the share is read into shared memory first, so that no copy waits for an address. The
// warps' states are merged through shared memory, and with several shares a second launch merges those.
constexpr int kDecStages = 4, kDecWarps = 4, kDecMaxPages = 512;
template <int kDim> struct DecodeSmem {
    static constexpr int kStride = kDim + 8;
    static constexpr int kPageBytes = kBlockTokens * kStride * 2;
    static constexpr int kRing = kDecWarps * kDecStages * kPageBytes, kRms = kDecWarps * kDecStages * kBlockTokens * 4;
    static constexpr int kMerge = kDecWarps * 16 * (kDim + 2) * 4;
    static constexpr int kBytes = (kRing + kRms + kDecMaxPages * 4) > kMerge ? (kRing + kRms + kDecMaxPages * 4) : kMerge;
};
template <int kDim>
__global__ void __launch_bounds__(128) shared_kv_decode_kernel(const AttendParams p) {
    using L = DecodeSmem<kDim>;
    constexpr int kK = kDim / 16;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    INGOT_PDL_TRIGGER();
    INGOT_PDL_WAIT();
    const int seq = blockIdx.z, kvh = blockIdx.y, group = p.n_head / p.n_head_kv;
    const int split = blockIdx.x % p.n_splits, row0 = blockIdx.x / p.n_splits * 16;  // rows: heads of the group
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j = lane & 3;
    const int pos = p.st.pos0[seq];
    const size_t tok = p.st.row_start[seq];
    const int page_a = p.map.page(p.map.first_visible(pos)), n_pages = p.map.page(pos) - page_a + 1;
    const int last_key = pos - p.map.first_visible(pos);  // keys 0..last_key of the chunk, 16 per page
    const int per = (n_pages + p.n_splits - 1) / p.n_splits, first = split * per, count = max(0, min(per, n_pages - first));
    const __half* rows = static_cast<const __half*>(p.rows);

    const uint32_t s_ring = (uint32_t)__cvta_generic_to_shared(smem_raw) + warp * kDecStages * L::kPageBytes;
    float* s_rms = reinterpret_cast<float*>(smem_raw + L::kRing) + warp * kDecStages * kBlockTokens;
    int* s_blk = reinterpret_cast<int*>(smem_raw + L::kRing + L::kRms);
    for (int i = threadIdx.x; i < count; i += 128)
        s_blk[i] = table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, page_a + first + i, p.status);
    __syncthreads();

    auto stage = [&](int i, int buf) {  // page i of the share
        if (i < count) {
            const int blk = s_blk[i];
            const __half* src = rows + ((size_t)max(blk, 0) * p.n_head_kv + kvh) * kBlockTokens * kDim;
            constexpr int kPieces = kDim / 8;
#pragma unroll
            for (int c = lane; c < kBlockTokens * kPieces; c += 32)
                cp16(s_ring + buf * L::kPageBytes + (c / kPieces * L::kStride + c % kPieces * 8) * 2, src + c * 8, blk >= 0);
            if (lane < 4) cp16((uint32_t)__cvta_generic_to_shared(s_rms + buf * kBlockTokens + lane * 4), p.inv_rms + (size_t)max(blk, 0) * kBlockTokens + lane * 4, blk >= 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int k = 0; k < kDecStages - 1; k++) stage(warp + k * kDecWarps, k);

    uint32_t qf[kK][4];
    {
        const __half* q = static_cast<const __half*>(p.q) + (tok * p.n_head + kvh * group) * kDim;
        const int lo = row0 + g, hi = lo + 8;
#pragma unroll
        for (int k = 0; k < kK; k++) {
            qf[k][0] = lo < group ? *reinterpret_cast<const uint32_t*>(q + (size_t)lo * kDim + k * 16 + 2 * j) : 0u;
            qf[k][1] = hi < group ? *reinterpret_cast<const uint32_t*>(q + (size_t)hi * kDim + k * 16 + 2 * j) : 0u;
            qf[k][2] = lo < group ? *reinterpret_cast<const uint32_t*>(q + (size_t)lo * kDim + k * 16 + 8 + 2 * j) : 0u;
            qf[k][3] = hi < group ? *reinterpret_cast<const uint32_t*>(q + (size_t)hi * kDim + k * 16 + 8 + 2 * j) : 0u;
        }
    }
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    float o[kDim / 8][4];
#pragma unroll
    for (int i = 0; i < kDim / 8; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const float scale = p.scale * 1.44269504f;

    int buf = 0;
    for (int i = warp; i < count; i += kDecWarps) {
        asm volatile("cp.async.wait_group %0;" ::"n"(kDecStages - 2) : "memory");
        __syncwarp();  // the page is in, and every lane is done with the buffer that is staged next
        stage(i + (kDecStages - 1) * kDecWarps, buf == 0 ? kDecStages - 1 : buf - 1);
        const uint32_t page = s_ring + buf * L::kPageBytes;
        const float* rms = s_rms + buf * kBlockTokens;
        float s[2][4];
#pragma unroll
        for (int e = 0; e < 4; e++) s[0][e] = s[1][e] = 0.f;
        const uint32_t a = page + (((lane & 7) + ((lane >> 4) & 1) * 8) * L::kStride + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
        for (int k = 0; k < kK; k++) {
            uint32_t b[4];
            ldmatrix4(b, a + k * 32);
            mma_16816(s[0], qf[k][0], qf[k][1], qf[k][2], qf[k][3], b[0], b[1]);
            mma_16816(s[1], qf[k][0], qf[k][1], qf[k][2], qf[k][3], b[2], b[3]);
        }
        const int left = last_key - (first + i) * kBlockTokens;  // keys of this page up to index `left` exist
        const bool held = s_blk[i] >= 0;
        float mx_lo = -INFINITY, mx_hi = -INFINITY;
#pragma unroll
        for (int nt = 0; nt < 2; nt++) {
            const float2 ks = *reinterpret_cast<const float2*>(rms + nt * 8 + 2 * j);
            const bool on0 = held && nt * 8 + 2 * j <= left, on1 = held && nt * 8 + 2 * j + 1 <= left;
            s[nt][0] = on0 ? s[nt][0] * (ks.x * scale) : -INFINITY;
            s[nt][1] = on1 ? s[nt][1] * (ks.y * scale) : -INFINITY;
            s[nt][2] = on0 ? s[nt][2] * (ks.x * scale) : -INFINITY;
            s[nt][3] = on1 ? s[nt][3] * (ks.y * scale) : -INFINITY;
            mx_lo = fmaxf(mx_lo, fmaxf(s[nt][0], s[nt][1]));
            mx_hi = fmaxf(mx_hi, fmaxf(s[nt][2], s[nt][3]));
        }
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
        const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);
        const float rf_lo = mn_lo == -INFINITY ? 0.f : mn_lo, rf_hi = mn_hi == -INFINITY ? 0.f : mn_hi;
        const float a_lo = exp2f(m_lo - rf_lo), a_hi = exp2f(m_hi - rf_hi);
        m_lo = mn_lo;
        m_hi = mn_hi;
        uint32_t pa[4];
        float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
        for (int nt = 0; nt < 2; nt++) {
            const float p0 = exp2f(s[nt][0] - rf_lo), p1 = exp2f(s[nt][1] - rf_lo), p2 = exp2f(s[nt][2] - rf_hi), p3 = exp2f(s[nt][3] - rf_hi);
            sum_lo += p0 + p1;
            sum_hi += p2 + p3;
            pa[nt * 2] = pack_half2_rn(p0, p1);
            pa[nt * 2 + 1] = pack_half2_rn(p2, p3);
        }
        l_lo = l_lo * a_lo + sum_lo;
        l_hi = l_hi * a_hi + sum_hi;
        if (__any_sync(0xffffffffu, a_lo != 1.f || a_hi != 1.f)) {
#pragma unroll
            for (int d = 0; d < kDim / 8; d++) { o[d][0] *= a_lo; o[d][1] *= a_lo; o[d][2] *= a_hi; o[d][3] *= a_hi; }
        }
        const uint32_t v = page + ((lane & 15) * L::kStride + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int d = 0; d < kDim / 16; d++) {
            uint32_t b[4];
            ldmatrix4_trans(b, v + d * 32);
            mma_16816(o[2 * d], pa[0], pa[1], pa[2], pa[3], b[0], b[1]);
            mma_16816(o[2 * d + 1], pa[0], pa[1], pa[2], pa[3], b[2], b[3]);
        }
        buf = buf + 1 == kDecStages ? 0 : buf + 1;
    }

    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);

    // merge the warps' states: [warp][16 rows][kDim] and (m, l)
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    float* so = reinterpret_cast<float*>(smem_raw);
    float* sml = so + kDecWarps * 16 * kDim;
#pragma unroll
    for (int i = 0; i < kDim / 8; i++) {
        *reinterpret_cast<float2*>(so + (warp * 16 + g) * kDim + i * 8 + 2 * j) = make_float2(o[i][0], o[i][1]);
        *reinterpret_cast<float2*>(so + (warp * 16 + g + 8) * kDim + i * 8 + 2 * j) = make_float2(o[i][2], o[i][3]);
    }
    if (j == 0) {
        sml[(warp * 16 + g) * 2] = m_lo; sml[(warp * 16 + g) * 2 + 1] = l_lo;
        sml[(warp * 16 + g + 8) * 2] = m_hi; sml[(warp * 16 + g + 8) * 2 + 1] = l_hi;
    }
    __syncthreads();
    const int rows_here = min(16, group - row0);
    for (int i = threadIdx.x; i < rows_here * kDim; i += 128) {
        const int r = i / kDim, d = i - r * kDim;
        float m = -INFINITY;
#pragma unroll
        for (int w = 0; w < kDecWarps; w++) m = fmaxf(m, sml[(w * 16 + r) * 2]);
        const float rf = m == -INFINITY ? 0.f : m;
        float l = 0.f, acc = 0.f;
#pragma unroll
        for (int w = 0; w < kDecWarps; w++) {
            const float f = exp2f(sml[(w * 16 + r) * 2] - rf);
            l = fmaf(f, sml[(w * 16 + r) * 2 + 1], l);
            acc = fmaf(f, so[(w * 16 + r) * kDim + d], acc);
        }
        const int h = kvh * group + row0 + r;
        const size_t row = tok;
        if (p.n_splits == 1) {
            if (d < p.out_dim) p.out.store(row, h * p.out_dim + d, acc / l);
        } else {
            float* part = p.part + ((row * p.n_head + h) * p.n_splits + split) * (kDim + 2);
            part[d] = acc;
            if (d == 0) { part[kDim] = m; part[kDim + 1] = l; }
        }
    }
}

// out = sum_s o_s 2^(m_s - M) / sum_s l_s 2^(m_s - M) over the splits of one (token, head)
__global__ void __launch_bounds__(128) shared_kv_merge_kernel(const AttendParams p) {
    INGOT_PDL_TRIGGER();
    INGOT_PDL_WAIT();
    const int h = blockIdx.x;
    const size_t row = blockIdx.y;
    const float* part = p.part + (row * p.n_head + h) * p.n_splits * (p.dim + 2);
    float m = -INFINITY;
    for (int s = 0; s < p.n_splits; s++) m = fmaxf(m, part[s * (p.dim + 2) + p.dim]);
    for (int d = threadIdx.x; d < p.out_dim; d += 128) {
        float l = 0.f, acc = 0.f;
        for (int s = 0; s < p.n_splits; s++) {
            const float f = exp2f(part[s * (p.dim + 2) + p.dim] - m);  // every query sees itself: the overall maximum is finite
            l = fmaf(f, part[s * (p.dim + 2) + p.dim + 1], l);
            acc = fmaf(f, part[s * (p.dim + 2) + d], acc);
        }
        p.out.store(row, h * p.out_dim + d, acc / l);
    }
}

template <int kDim>
int launch_mma(ingot_skv* kv, AttendParams p, cudaStream_t s) {
    const int group = p.n_head / p.n_head_kv;
    if (p.st.max_len > 1) {
        constexpr int kSmem = 2 * (MmaTile<kDim>::kBytes + kTileKeys * 8);
        const dim3 grid((unsigned)(((size_t)p.st.max_len * group + 127) / 128), p.n_head_kv, p.st.n_seq);
        p.n_splits = 1;
        INGOT_CUDA_TRY(cudaFuncSetAttribute(shared_kv_mma_kernel<kDim>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem));
        INGOT_CUDA_TRY(ingot_launch_pdl(shared_kv_mma_kernel<kDim>, grid, dim3(256), kSmem, s, p));
        return INGOT_OK;
    }
    // Shares of the keys: CTAs run in rounds of as many as fit the GPU, and a share costs about 64 keys' time besides its keys, so
    // the count that minimises rounds * (share + 64) - and never more pages per share than the kernel's table holds.
    const int row_tiles = (group + 15) / 16, keys = p.max_blocks * kBlockTokens;
    const int ctas = row_tiles * p.n_head_kv * p.st.n_seq, slots = kv->num_sms * std::max(1, std::min(4, 220 * 1024 / DecodeSmem<kDim>::kBytes));
    long long best = -1;
    for (int n = 1; n <= 64; n++) {
        const int share = (keys + n - 1) / n;
        if (n > 1 && share < kSplitKeysMin) break;
        const long long cost = ((long long)ctas * n + slots - 1) / slots * (share + 64);
        if (best < 0 || cost < best) { best = cost; p.n_splits = n; }
    }
    p.n_splits = std::max(p.n_splits, (p.max_blocks + kDecMaxPages - 1) / kDecMaxPages);
    if (p.n_splits > 1) {
        const size_t need = (size_t)p.st.n_tok * p.n_head * p.n_splits * (kDim + 2);
        if (need > kv->part_floats) {
            float* fresh = nullptr;
            INGOT_CUDA_TRY(cudaMalloc(&fresh, need * sizeof(float)));
            if (kv->part) kv->retired.push_back(kv->part);  // a captured graph may still point into it
            kv->part = fresh;
            kv->part_floats = need;
        }
        p.part = kv->part;
    }
    INGOT_CUDA_TRY(cudaFuncSetAttribute(shared_kv_decode_kernel<kDim>, cudaFuncAttributeMaxDynamicSharedMemorySize, DecodeSmem<kDim>::kBytes));
    const dim3 grid(row_tiles * p.n_splits, p.n_head_kv, p.st.n_seq);
    INGOT_CUDA_TRY(ingot_launch_pdl(shared_kv_decode_kernel<kDim>, grid, dim3(128), size_t(DecodeSmem<kDim>::kBytes), s, p));
    if (p.n_splits > 1) INGOT_CUDA_TRY(ingot_launch_pdl(shared_kv_merge_kernel, dim3(p.n_head, p.st.n_tok), dim3(128), 0, s, p));
    return INGOT_OK;
}

int create(ingot_skv** out, int n_layer, int n_head_kv, int head_dim, int dtype, int chunk, int window, int n_blocks, bool scales, bool tiles, const char* who) {
    *out = nullptr;
    INGOT_REQUIRE(n_layer >= 1 && n_head_kv >= 1 && n_blocks >= 1 && chunk >= 0 && window >= 0, std::string(who) + ": bad sizes");
    INGOT_REQUIRE(dtype == INGOT_F32 || dtype == INGOT_F16, std::string(who) + ": rows are f32 or f16");
    const int longest = scales ? 512 : 1024;
    if (head_dim < 4 || head_dim > longest || head_dim % 4 != 0) {
        ingot_set_error(std::string(who) + ": row length must be a multiple of 4 and at most " + std::to_string(longest));
        return INGOT_ERR_UNSUPPORTED;
    }
    ingot_skv* kv = new (std::nothrow) ingot_skv();
    if (!kv) return INGOT_ERR_NOMEM;
    kv->n_layer = n_layer; kv->n_head_kv = n_head_kv; kv->dim = head_dim; kv->dtype = dtype; kv->chunk = chunk; kv->window = window; kv->n_blocks = n_blocks;
    kv->tiled = tiles && dtype == INGOT_F16 && head_dim % 64 == 0;
    kv->layer_elems = (size_t)n_blocks * n_head_kv * kBlockTokens * head_dim;
    const size_t bytes = kv->layer_elems * n_layer * (dtype == INGOT_F32 ? 4 : 2), scale_bytes = (size_t)n_layer * n_blocks * kBlockTokens * 4;
    cudaError_t e;
    // zero-filled: rows that were never written stay finite, so a masked key cannot inject NaN through 0 * garbage
    if ((e = cudaGetDevice(&kv->device)) != cudaSuccess || (e = cudaDeviceGetAttribute(&kv->num_sms, cudaDevAttrMultiProcessorCount, kv->device)) != cudaSuccess ||
        (e = cudaMalloc(&kv->rows, bytes)) != cudaSuccess || (e = cudaMalloc(&kv->status_dev, sizeof(int))) != cudaSuccess ||
        (e = cudaMemset(kv->rows, 0, bytes)) != cudaSuccess || (e = cudaMemset(kv->status_dev, 0, sizeof(int))) != cudaSuccess ||
        (scales && ((e = cudaMalloc(&kv->inv_rms, scale_bytes)) != cudaSuccess || (e = cudaMemset(kv->inv_rms, 0, scale_bytes)) != cudaSuccess)) ||
        (e = cudaDeviceSynchronize()) != cudaSuccess) {
        const int rc = ingot_cuda_fail(e, who);
        ingot_skv_destroy(kv);
        return rc;
    }
    *out = kv;
    return INGOT_OK;
}

bool step_ok(const ingot_step* st) {
    return st && st->n_tok >= 1 && st->n_seq >= 1 && st->n_seq <= 65535 && st->max_len >= 1 && st->row_seq && st->row_start && st->len && st->pos0;
}

}  // namespace

int launch_shared_kv_plain(const AttendParams& p, int dtype, cudaStream_t stream) {
    return dtype == INGOT_F32 ? launch_plain<float>(p, stream) : launch_plain<__half>(p, stream);
}

extern "C" {

int ingot_skv_create(ingot_skv** out, int n_layer, int n_head_kv, int head_dim, int dtype, int chunk, int n_blocks) {
    INGOT_REQUIRE(out != nullptr, "ingot_skv_create: out is null");
    return create(out, n_layer, n_head_kv, head_dim, dtype, chunk, 0, n_blocks, true, false, "ingot_skv_create");
}

int ingot_skv_create_window(ingot_skv** out, int n_layer, int n_head_kv, int row_length, int dtype, int window, int n_blocks) {
    INGOT_REQUIRE(out != nullptr, "ingot_skv_create_window: out is null");
    return create(out, n_layer, n_head_kv, row_length, dtype, 0, window, n_blocks, false, true, "ingot_skv_create_window");
}

int ingot_skv_create_joined(ingot_skv** out, int n_layer, int n_head_kv, int row_length, int dtype, int window, int n_blocks) {
    INGOT_REQUIRE(out != nullptr, "ingot_skv_create_joined: out is null");
    return create(out, n_layer, n_head_kv, row_length, dtype, 0, window, n_blocks, false, false, "ingot_skv_create_joined");
}

void ingot_skv_destroy(ingot_skv* kv) {
    if (!kv) return;
    cudaFree(kv->rows);
    cudaFree(kv->inv_rms);
    cudaFree(kv->status_dev);
    cudaFree(kv->part);
    for (void* p : kv->retired) cudaFree(p);
    delete kv;
}

int ingot_skv_pages(int chunk, int n_positions) {
    if (n_positions < 1 || chunk < 0) return 0;
    const PageMap map = {chunk, (chunk + kBlockTokens - 1) / kBlockTokens, 0};
    return map.page(n_positions - 1) + 1;
}

int* ingot_skv_status_dev(ingot_skv* kv) { return kv ? kv->status_dev : nullptr; }

int ingot_skv_row_length(int head_size) {
    if (head_size < 1) return 0;
    for (int d : {32, 64, 96, 128, 192, 256})
        if (head_size <= d) return d;
    return (head_size + 15) / 16 * 16;
}

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
    INGOT_REQUIRE(kv->inv_rms, "ingot_skv_append: the cache was created for rows without scales");
    INGOT_REQUIRE_DEVICE(kv);
    INGOT_REQUIRE(layer >= 0 && layer < kv->n_layer, "ingot_skv_append: layer out of range");
    INGOT_REQUIRE(proj_dev && q_norm_dev && k_norm_dev && q_out_dev && tables_dev && max_blocks >= 1, "ingot_skv_append: null argument");
    INGOT_REQUIRE(proj_ld % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0, "ingot_skv_append: rows and offsets must be multiples of 4 floats");
    INGOT_REQUIRE(n_head >= kv->n_head_kv && n_head % kv->n_head_kv == 0, "ingot_skv_append: n_head must be a multiple of n_head_kv");
    INGOT_REQUIRE(head_size >= 1 && head_size <= kv->dim, "ingot_skv_append: head size beyond the row length");
    const size_t esz = kv->dtype == INGOT_F32 ? 4 : 2;
    AppendParams p = {*step, proj_dev, proj_ld, q_off, k_off, n_head, kv->n_head_kv, kv->dim, n_head * head_size, kv->n_head_kv * head_size,
                      q_norm_dev, k_norm_dev, eps, q_out_dev, static_cast<char*>(kv->rows) + kv->layer_elems * layer * esz,
                      kv->inv_rms + (size_t)layer * kv->n_blocks * kBlockTokens, tables_dev, first_page_dev, max_blocks, kv->n_blocks,
                      page_map(kv), kv->status_dev};
    auto kernel = kv->dtype == INGOT_F32 ? shared_kv_append_kernel<float> : shared_kv_append_kernel<__half>;
    INGOT_CUDA_TRY(ingot_launch_pdl(kernel, dim3(step->n_tok), dim3(kAppendThreads), 0, static_cast<cudaStream_t>(stream), p));
    return INGOT_OK;
}

int ingot_skv_attend(ingot_skv* kv, int layer, const ingot_step* step, const void* q_dev, int n_head, int out_dim, float scale,
                     float out_scale, const ingot_act_out* out, const int32_t* tables_dev, const int32_t* first_page_dev, int max_blocks, int impl, void* stream) {
    INGOT_REQUIRE(kv && step_ok(step), "ingot_skv_attend: null handle or bad step");
    INGOT_REQUIRE(kv->inv_rms, "ingot_skv_attend: the cache was created for rows without scales");
    INGOT_REQUIRE_DEVICE(kv);
    INGOT_REQUIRE(layer >= 0 && layer < kv->n_layer, "ingot_skv_attend: layer out of range");
    INGOT_REQUIRE(q_dev && out && tables_dev && max_blocks >= 1, "ingot_skv_attend: null argument");
    INGOT_REQUIRE(n_head >= kv->n_head_kv && n_head % kv->n_head_kv == 0, "ingot_skv_attend: n_head must be a multiple of n_head_kv");
    INGOT_REQUIRE(out_dim >= 1 && out_dim <= kv->dim, "ingot_skv_attend: bad output");
    const size_t esz = kv->dtype == INGOT_F32 ? 4 : 2;
    AttendParams p = {*step, q_dev, static_cast<const char*>(kv->rows) + kv->layer_elems * layer * esz,
                      kv->inv_rms + (size_t)layer * kv->n_blocks * kBlockTokens, tables_dev, first_page_dev, max_blocks, kv->n_blocks, n_head, kv->n_head_kv,
                      kv->dim, out_dim, page_map(kv), scale,
                      SharedOut{out->f32, static_cast<__nv_bfloat16*>(out->hi), static_cast<__nv_bfloat16*>(out->lo), out->ld, out_scale}, kv->status_dev, 1, nullptr};
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (kv->dtype == INGOT_F32) return launch_plain<float>(p, s);
    // portions of prompts over rows of 128 values: the tcgen05 kernel, from 256 (token, head) rows per KV head on
    if (kv->dim == 128 && (impl == 3 || (impl == 0 && (long long)step->max_len * (n_head / kv->n_head_kv) >= 256))) {
        const int rc = launch_shared_kv_sm100(kv, layer, p, s);
        if (rc != INGOT_ERR_UNSUPPORTED || impl == 3) return rc;
    }
    if (impl != 1) switch (kv->dim) {
        case 32: return launch_mma<32>(kv, p, s);
        case 64: return launch_mma<64>(kv, p, s);
        case 96: return launch_mma<96>(kv, p, s);
        case 128: return launch_mma<128>(kv, p, s);
        case 192: return launch_mma<192>(kv, p, s);
        case 256: return launch_mma<256>(kv, p, s);
        default: break;
    }
    return launch_plain<__half>(p, s);
}

}  // extern "C"
