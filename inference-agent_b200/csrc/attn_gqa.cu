// Grouped-query attention over joined rows: one cached row per token and KV head, [key | value] side by side, heads of any size.
// No counterpart in the reference beyond its plain form (one head size, RoPE in halves, no norms, windows, sinks or gates).
//
// What a layer may have, each of it a parameter:
//   query / key norm   none; RMS over a head with one weight for all of them; RMS over the whole projection
//   rotation           the first rot_dims values of a head in neighbouring pairs (2 i, 2 i + 1), by position * turns[i] full turns, cosine and
//                      sine times a gain; the angle is reduced to a fraction of a turn in double precision
//   value mixing       v <- (1 - mix) v + mix v_first with the values of the same token in an earlier layer; the cache gets the mixed ones
//   visibility         causal, or a window that slides along (PageMap)
//   sink               one more term exp(sink_h) in a head's softmax sum
//   gate               the result times sigmoid(z), z one number per head or per value, read from the projection row
//
// The cache is the window form of attn_shared_kv.cuh in plain page order, [page][kv head][16][dim | vdim]. Three kernels attend: portions
// of prompts on tcgen05 (attn_gqa_sm100.cu); decoded tokens and short portions on warp-level MMAs, the keys split over CTAs (here); any
// size in f32 arithmetic (the plain kernel of attn_shared_kv.cu).
#include <algorithm>
#include <cstdlib>

#include "attn_shared_kv.cuh"
#include "sm100_ptx.cuh"

namespace {

using namespace ingot_sm100;

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float clamp_half(float v) { return fminf(fmaxf(v, -65504.f), 65504.f); }
__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__half* p, float4 v) {
    const __half2 h[2] = {__floats2half2_rn(clamp_half(v.x), clamp_half(v.y)), __floats2half2_rn(clamp_half(v.z), clamp_half(v.w))};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(h);
}
__device__ __forceinline__ float dot4(float4 v, float acc) {
    return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, acc))));
}

constexpr int kMaxRot = 1024;  // rotated values per head
constexpr int kAppendThreads = 256;

// A warp per head, one CTA or a few per token: queries out, keys and values into the cache.
struct AppendParams {
    ingot_step st;
    const float* proj;
    int proj_ld, q_off, k_off, v_off;
    ingot_gqa_shape sh;
    const float *q_norm, *k_norm;
    float eps;
    const double* turns;
    float rot_gain;
    float* first_values;  // [n_tok][n_head_kv * vdim]; null: values are not mixed
    int store_first;      // this layer's values are the first ones
    float mix;
    void* q_out;
    void* rows;
    const int32_t *tables, *first_page;
    int max_blocks, n_blocks;
    PageMap map;
    int* status;
};

template <typename T>
__global__ void __launch_bounds__(kAppendThreads) gqa_append_kernel(const AppendParams p) {
    INGOT_PDL_TRIGGER();
    __shared__ float red[2 * kAppendThreads / 32], s_cos[kMaxRot / 2], s_sin[kMaxRot / 2];
    const int tok = blockIdx.x, seq = p.st.row_seq[tok], warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos = p.st.pos0[seq] + tok - p.st.row_start[seq];
    const int dim = p.sh.dim, vdim = p.sh.vdim, rot = p.sh.rot_dims, H = p.sh.n_head, G = p.sh.n_head_kv;
    for (int i = threadIdx.x; i < rot / 2; i += kAppendThreads) {
        double t = double(pos) * p.turns[i];
        t -= rint(t);
        float c, s;
        sincospif(2.0f * float(t), &s, &c);
        s_cos[i] = c * p.rot_gain;
        s_sin[i] = s * p.rot_gain;
    }
    INGOT_PDL_WAIT();
    const float* row = p.proj + (size_t)tok * p.proj_ld;
    float inv_q = 1.f, inv_k = 1.f;
    if (p.sh.norm == INGOT_QK_NORM_ALL) {
        float sq = 0.f, sk = 0.f;
        for (int i = threadIdx.x * 4; i < H * dim; i += kAppendThreads * 4) sq = dot4(*reinterpret_cast<const float4*>(row + p.q_off + i), sq);
        for (int i = threadIdx.x * 4; i < G * dim; i += kAppendThreads * 4) sk = dot4(*reinterpret_cast<const float4*>(row + p.k_off + i), sk);
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        if (lane == 0) { red[warp] = sq; red[kAppendThreads / 32 + warp] = sk; }
    }
    __syncthreads();
    if (p.sh.norm == INGOT_QK_NORM_ALL) {
        float sq = 0.f, sk = 0.f;
#pragma unroll
        for (int w = 0; w < kAppendThreads / 32; w++) { sq += red[w]; sk += red[kAppendThreads / 32 + w]; }
        inv_q = 1.0f / sqrtf(sq / float(H * p.sh.dim_count) + p.eps);
        inv_k = 1.0f / sqrtf(sk / float(G * p.sh.dim_count) + p.eps);
    }
    const int blk = table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, p.map.page(pos), p.status);
    T* page = static_cast<T*>(p.rows) + ((size_t)max(blk, 0) * G * kBlockTokens + p.map.slot(pos)) * (dim + vdim);  // of KV head 0
    const size_t head_stride = (size_t)kBlockTokens * (dim + vdim);
    for (int h = blockIdx.y * (kAppendThreads / 32) + warp; h < H + G; h += gridDim.y * (kAppendThreads / 32)) {
        const bool is_q = h < H;
        const float* src = row + (is_q ? p.q_off + h * dim : p.k_off + (h - H) * dim);
        const float* w = is_q ? p.q_norm : p.k_norm;
        float inv = is_q ? inv_q : inv_k;
        if (p.sh.norm == INGOT_QK_NORM_HEAD) {
            float ss = 0.f;
            for (int d = lane * 4; d < dim; d += 128) ss = dot4(*reinterpret_cast<const float4*>(src + d), ss);
            inv = 1.0f / sqrtf(warp_sum(ss) / float(p.sh.dim_count) + p.eps);
        } else if (p.sh.norm == INGOT_QK_NORM_ALL) {
            w += (is_q ? h : h - H) * dim;
        }
        T* dst = is_q ? static_cast<T*>(p.q_out) + ((size_t)tok * H + h) * dim : page + (h - H) * head_stride;
        if (!is_q && blk < 0) continue;
        for (int d = lane * 4; d < dim; d += 128) {
            float4 v = *reinterpret_cast<const float4*>(src + d);
            if (p.sh.norm != INGOT_QK_NORM_NONE) {
                const float4 g = *reinterpret_cast<const float4*>(w + d);
                v.x *= inv * g.x; v.y *= inv * g.y; v.z *= inv * g.z; v.w *= inv * g.w;
            }
            if (d < rot) {
                const float c = s_cos[d / 2], s = s_sin[d / 2], x = v.x;
                v.x = x * c - v.y * s;
                v.y = v.y * c + x * s;
            }
            if (d + 2 < rot) {
                const float c = s_cos[d / 2 + 1], s = s_sin[d / 2 + 1], x = v.z;
                v.z = x * c - v.w * s;
                v.w = v.w * c + x * s;
            }
            put4(dst + d, v);
        }
    }
    const float keep = 1.0f - p.mix;
    for (int i = (blockIdx.y * kAppendThreads + threadIdx.x) * 4; i < G * vdim; i += gridDim.y * kAppendThreads * 4) {
        float4 v = *reinterpret_cast<const float4*>(row + p.v_off + i);
        if (p.first_values) {
            float4* f = reinterpret_cast<float4*>(p.first_values + (size_t)tok * G * vdim + i);
            if (p.store_first) {
                *f = v;
            } else {
                const float4 u = *f;
                v = make_float4(fmaf(p.mix, u.x, keep * v.x), fmaf(p.mix, u.y, keep * v.y), fmaf(p.mix, u.z, keep * v.z), fmaf(p.mix, u.w, keep * v.w));
            }
        }
        if (blk >= 0) put4(page + i / vdim * head_stride + dim + i % vdim, v);
    }
}

// ---- decoded tokens and short portions: f16, m16n8k16 MMAs, the keys split over CTAs ---------------------------------------------------
// A CTA serves 16 (token, head) rows of one KV head of one sequence over one share of the pages they see. Its four warps take every fourth
// page each through a ring of bulk copies of their own - a lane fetches a slot's row, no barrier in the key loop - the block table of the
// share is in shared memory first, so that no copy waits for an address. The warps' states are merged through shared memory; several shares
// are merged by a second launch. kMax: most columns of a key or a value; the loops over 16-column steps stop at the true sizes.
// Waits for copies are bounded: a warp that gives up waits, again bounded, for those in flight and raises the status word.
constexpr unsigned long long kWaitLimitNs = 2000000000ull;
constexpr int kMaxRing = 3, kWarps = 4, kMaxSharePages = 1024, kMaxSplits = 64, kSplitKeysMin = 128;
constexpr int kSmemLimit = 227 * 1024;
struct GqaSmem {
    int stride, page_bytes, blocks, bytes;  // stride: halves between rows, 16 bytes past the row so that ldmatrix has no bank conflicts
    int ring;                             // pages per warp: three, or two where that lets two CTAs share an SM
    __host__ __device__ GqaSmem(int row, int vdim, int share_pages) {
        stride = row + 8;
        page_bytes = kBlockTokens * stride * 2;
        ring = kWarps * kMaxRing * page_bytes <= 104 * 1024 ? kMaxRing : 2;
        blocks = kWarps * ring * page_bytes;
        const int loop = blocks + share_pages * 4, merge = kWarps * 16 * (vdim + 2) * 4;
        bytes = loop > merge ? loop : merge;
    }
};
__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <int kMax>
__global__ void __launch_bounds__(kWarps * 32) gqa_mma_kernel(const AttendParams p, int share_pages) {
    constexpr int kK = kMax / 16, kN = kMax / 8;
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ uint64_t s_full[kWarps][kMaxRing];
    __shared__ uint32_t s_abort;
    INGOT_PDL_TRIGGER();
    INGOT_PDL_WAIT();
    const int seq = blockIdx.z, kvh = blockIdx.y, group = p.n_head / p.n_head_kv, n_rows = p.st.len[seq] * group;
    const int split = blockIdx.x % p.n_splits, row0 = blockIdx.x / p.n_splits * 16;
    if (row0 >= n_rows) return;
    const GqaSmem L(p.dim, p.out_dim, share_pages);
    const int ring = L.ring;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j = lane & 3;
    const int pos0 = p.st.pos0[seq], n_k = p.q_dim / 16, n_v = p.out_dim / 16;
    const size_t tok0 = p.st.row_start[seq];
    const int pos_first = pos0 + row0 / group, pos_last = pos0 + (min(row0 + 16, n_rows) - 1) / group;
    const int page_a = p.map.page(p.map.first_visible(pos_first)), n_pages = p.map.page(pos_last) - page_a + 1;
    const int per = (n_pages + p.n_splits - 1) / p.n_splits, first = split * per, count = max(0, min(min(per, share_pages), n_pages - first));
    const __half* rows = static_cast<const __half*>(p.rows);
    const uint32_t s_ring = (uint32_t)__cvta_generic_to_shared(smem) + warp * ring * L.page_bytes;
    int* s_blk = reinterpret_cast<int*>(smem + L.blocks);
    for (int i = threadIdx.x; i < count; i += kWarps * 32)
        s_blk[i] = table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, page_a + first + i, p.status);
    if (threadIdx.x == 0) s_abort = 0;
    if (lane < ring) mbar_init(smem_u32(&s_full[warp][lane]), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    __syncthreads();

    const uint32_t row_bytes = p.dim * 2;
    auto stage = [&](int i, int buf) {  // page i of the share; one without a block comes from block 0 and is masked
        if (i >= count) return;
        const uint32_t full = smem_u32(&s_full[warp][buf]);
        if (lane == 0) mbar_expect_tx(full, kBlockTokens * row_bytes);
        __syncwarp();
        if (lane < kBlockTokens)
            bulk_load(s_ring + buf * L.page_bytes + lane * L.stride * 2, rows + (((size_t)max(s_blk[i], 0) * p.n_head_kv + kvh) * kBlockTokens + lane) * p.dim, row_bytes, full);
    };
    for (int k = 0; k < ring - 1; k++) stage(warp + k * kWarps, k);

    const int r_lo = row0 + g, r_hi = r_lo + 8;
    const int pos_lo = pos0 + min(r_lo, n_rows - 1) / group, pos_hi = pos0 + min(r_hi, n_rows - 1) / group;
    const int vis_lo = p.map.first_visible(pos_lo), vis_hi = p.map.first_visible(pos_hi);
    uint32_t qf[kK][4];
    {
        const __half* q = static_cast<const __half*>(p.q);
        const __half* a = q + ((tok0 + r_lo / group) * p.n_head + kvh * group + r_lo % group) * p.q_dim;
        const __half* b = q + ((tok0 + r_hi / group) * p.n_head + kvh * group + r_hi % group) * p.q_dim;
#pragma unroll
        for (int k = 0; k < kK; k++) {
            const bool lo = k < n_k && r_lo < n_rows, hi = k < n_k && r_hi < n_rows;
            qf[k][0] = lo ? *reinterpret_cast<const uint32_t*>(a + k * 16 + 2 * j) : 0u;
            qf[k][1] = hi ? *reinterpret_cast<const uint32_t*>(b + k * 16 + 2 * j) : 0u;
            qf[k][2] = lo ? *reinterpret_cast<const uint32_t*>(a + k * 16 + 8 + 2 * j) : 0u;
            qf[k][3] = hi ? *reinterpret_cast<const uint32_t*>(b + k * 16 + 8 + 2 * j) : 0u;
        }
    }
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    float o[kN][4];
#pragma unroll
    for (int i = 0; i < kN; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const float scale = p.scale * 1.44269504f;

    const int vis_max = p.map.first_visible(pos_last);
    int buf = 0, round = 0;
    for (int i = warp; i < count; i += kWarps) {
        const bool ok = mbar_wait(smem_u32(&s_full[warp][buf]), round & 1, &s_abort, kWaitLimitNs);
        if (!__all_sync(0xffffffffu, ok)) {
            for (int k = i, b = buf, r = round; k < min(count, i + (ring - 1) * kWarps); k += kWarps) {  // what is in flight must land first
                const uint64_t t0 = globaltimer_ns();
                while (!mbar_try_wait(smem_u32(&s_full[warp][b]), r & 1) && globaltimer_ns() - t0 < 100000000ull) {}
                if (++b == ring) { b = 0; r++; }
            }
            break;
        }
        // every lane is done with the buffer that is staged next: the votes above came after its last use
        stage(i + (ring - 1) * kWarps, buf == 0 ? ring - 1 : buf - 1);
        const uint32_t page = s_ring + buf * L.page_bytes;
        float s[2][4], s2[2][4];
#pragma unroll
        for (int e = 0; e < 4; e++) s[0][e] = s[1][e] = s2[0][e] = s2[1][e] = 0.f;
        const uint32_t a = page + (((lane & 7) + ((lane >> 4) & 1) * 8) * L.stride + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
        for (int k = 0; k < kK; k += 2) {  // even and odd steps in sums of their own: shorter chains
            if (k >= n_k) break;
            uint32_t b[4];
            ldmatrix4(b, a + k * 32);
            mma_16816(s[0], qf[k][0], qf[k][1], qf[k][2], qf[k][3], b[0], b[1]);
            mma_16816(s[1], qf[k][0], qf[k][1], qf[k][2], qf[k][3], b[2], b[3]);
            if (k + 1 >= n_k) break;
            ldmatrix4(b, a + k * 32 + 32);
            mma_16816(s2[0], qf[k + 1][0], qf[k + 1][1], qf[k + 1][2], qf[k + 1][3], b[0], b[1]);
            mma_16816(s2[1], qf[k + 1][0], qf[k + 1][1], qf[k + 1][2], qf[k + 1][3], b[2], b[3]);
        }
#pragma unroll
        for (int e = 0; e < 4; e++) {
            s[0][e] = (s[0][e] + s2[0][e]) * scale;
            s[1][e] = (s[1][e] + s2[1][e]) * scale;
        }
        const int key_first = (page_a + first + i) * kBlockTokens;
        if (key_first < vis_max || key_first + kBlockTokens - 1 > pos_first || s_blk[i] < 0) {  // some row does not see all of the page
            const bool held = s_blk[i] >= 0;
#pragma unroll
            for (int nt = 0; nt < 2; nt++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int key = key_first + 2 * j + nt * 8 + e;
                    if (!held || key < vis_lo || key > pos_lo) s[nt][e] = -INFINITY;
                    if (!held || key < vis_hi || key > pos_hi) s[nt][2 + e] = -INFINITY;
                }
        }
        float mx_lo = fmaxf(fmaxf(s[0][0], s[0][1]), fmaxf(s[1][0], s[1][1])), mx_hi = fmaxf(fmaxf(s[0][2], s[0][3]), fmaxf(s[1][2], s[1][3]));
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
        const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);
        // a row that has not seen a key yet keeps -inf; 0 stands in for it in the exponents
        const float rf_lo = mn_lo == -INFINITY ? 0.f : mn_lo, rf_hi = mn_hi == -INFINITY ? 0.f : mn_hi;
        const float a_lo = ex2(m_lo - rf_lo), a_hi = ex2(m_hi - rf_hi);
        m_lo = mn_lo;
        m_hi = mn_hi;
        uint32_t pa[4];
        float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
        for (int nt = 0; nt < 2; nt++) {
            const float p0 = ex2(s[nt][0] - rf_lo), p1 = ex2(s[nt][1] - rf_lo), p2 = ex2(s[nt][2] - rf_hi), p3 = ex2(s[nt][3] - rf_hi);
            sum_lo += p0 + p1;
            sum_hi += p2 + p3;
            pa[nt * 2] = pack_half2_rn(p0, p1);
            pa[nt * 2 + 1] = pack_half2_rn(p2, p3);
        }
        l_lo = l_lo * a_lo + sum_lo;
        l_hi = l_hi * a_hi + sum_hi;
        if (__any_sync(0xffffffffu, a_lo != 1.f || a_hi != 1.f)) {
#pragma unroll
            for (int d = 0; d < kN; d++) { o[d][0] *= a_lo; o[d][1] *= a_lo; o[d][2] *= a_hi; o[d][3] *= a_hi; }
        }
        const uint32_t v = page + ((lane & 15) * L.stride + p.v_off + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int d = 0; d < kN / 2; d++) {
            if (d >= n_v) break;
            uint32_t b[4];
            ldmatrix4_trans(b, v + d * 32);
            mma_16816(o[2 * d], pa[0], pa[1], pa[2], pa[3], b[0], b[1]);
            mma_16816(o[2 * d + 1], pa[0], pa[1], pa[2], pa[3], b[2], b[3]);
        }
        if (++buf == ring) { buf = 0; round++; }
    }

    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);

    // merge the warps' states: [warp][16 rows][out_dim] and (m, l)
    __syncthreads();
    if (threadIdx.x == 0 && s_abort) atomicOr(p.status, kDevErrBarrierTimeout);
    const int dv = p.out_dim;
    float* so = reinterpret_cast<float*>(smem);
    float* sml = so + kWarps * 16 * dv;
#pragma unroll
    for (int i = 0; i < kN; i++) {
        if (i >= 2 * n_v) break;
        *reinterpret_cast<float2*>(so + (warp * 16 + g) * dv + i * 8 + 2 * j) = make_float2(o[i][0], o[i][1]);
        *reinterpret_cast<float2*>(so + (warp * 16 + g + 8) * dv + i * 8 + 2 * j) = make_float2(o[i][2], o[i][3]);
    }
    if (j == 0) {
        sml[(warp * 16 + g) * 2] = m_lo; sml[(warp * 16 + g) * 2 + 1] = l_lo;
        sml[(warp * 16 + g + 8) * 2] = m_hi; sml[(warp * 16 + g + 8) * 2 + 1] = l_hi;
    }
    __syncthreads();
    const int rows_here = min(16, n_rows - row0);
    for (int i = threadIdx.x * 2; i < rows_here * dv; i += kWarps * 64) {
        const int r = i / dv, d = i - r * dv, h = kvh * group + (row0 + r) % group;
        const size_t row = tok0 + (row0 + r) / group;
        float m = -INFINITY;
#pragma unroll
        for (int w = 0; w < kWarps; w++) m = fmaxf(m, sml[(w * 16 + r) * 2]);
        const float sink = p.n_splits == 1 && p.sink ? p.sink[h] * 1.44269504f : -INFINITY;
        m = fmaxf(m, sink);
        const float rf = m == -INFINITY ? 0.f : m;
        float l = exp2f(sink - rf), x = 0.f, y = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; w++) {
            const float f = exp2f(sml[(w * 16 + r) * 2] - rf);
            const float2 v = *reinterpret_cast<const float2*>(so + (w * 16 + r) * dv + d);
            l = fmaf(f, sml[(w * 16 + r) * 2 + 1], l);
            x = fmaf(f, v.x, x);
            y = fmaf(f, v.y, y);
        }
        if (p.n_splits == 1) {
            const float inv = 1.0f / l;
            p.out.store2(row, h * dv + d, x * inv * p.gate.at(row, h, dv, d), y * inv * p.gate.at(row, h, dv, d + 1));
        } else {
            float* part = p.part + ((row * p.n_head + h) * p.n_splits + split) * (dv + 2);
            *reinterpret_cast<float2*>(part + d) = make_float2(x, y);
            if (d == 0) { part[dv] = m; part[dv + 1] = l; }
        }
    }
}

// out = gate * sum_s o_s 2^(m_s - M) / (sum_s l_s 2^(m_s - M) + 2^(sink - M)) over the shares of one (token, head)
__global__ void __launch_bounds__(128) gqa_merge_kernel(const AttendParams p) {
    INGOT_PDL_TRIGGER();
    INGOT_PDL_WAIT();
    __shared__ float s_f[kMaxSplits], s_m[kMaxSplits], s_l[kMaxSplits];
    const int h = blockIdx.x, dv = p.out_dim, ld = dv + 2, seq = blockIdx.z;
    if ((int)blockIdx.y >= p.st.len[seq]) return;
    const size_t row = (size_t)p.st.row_start[seq] + blockIdx.y;
    const float* part = p.part + (row * p.n_head + h) * p.n_splits * ld;
    const float sink = p.sink ? p.sink[h] * 1.44269504f : -INFINITY;
    if (threadIdx.x < p.n_splits) {
        const float2 ml = *reinterpret_cast<const float2*>(part + threadIdx.x * ld + dv);
        s_m[threadIdx.x] = ml.x;
        s_l[threadIdx.x] = ml.y;
    }
    __syncthreads();
    float top = sink;  // every query sees itself: the overall maximum is finite
    for (int s = 0; s < p.n_splits; s++) top = fmaxf(top, s_m[s]);
    if (threadIdx.x < p.n_splits) s_f[threadIdx.x] = exp2f(s_m[threadIdx.x] - top);
    __syncthreads();
    float l = exp2f(sink - top);
    for (int s = 0; s < p.n_splits; s++) l = fmaf(s_f[s], s_l[s], l);
    const float inv = 1.0f / l;
    for (int d = threadIdx.x * 2; d < dv; d += 256) {
        float a = 0.f, b = 0.f;
#pragma unroll 8
        for (int s = 0; s < p.n_splits; s++) {
            const float2 v = *reinterpret_cast<const float2*>(part + s * ld + d);
            a = fmaf(s_f[s], v.x, a);
            b = fmaf(s_f[s], v.y, b);
        }
        p.out.store2(row, h * dv + d, a * inv * p.gate.at(row, h, dv, d), b * inv * p.gate.at(row, h, dv, d + 1));
    }
}

bool mma_takes(int dim, int vdim) { return dim % 16 == 0 && vdim % 16 == 0 && dim <= 256 && vdim <= 256; }

int launch_mma(ingot_skv* kv, AttendParams p, cudaStream_t s) {
    const int group = p.n_head / p.n_head_kv, row_tiles = (p.st.max_len * group + 15) / 16;
    const int pages = p.map.window > 0 ? std::min(p.max_blocks, (p.map.window + p.st.max_len + 2 * kBlockTokens) / kBlockTokens) : p.max_blocks;
    // Shares of the keys: CTAs run in rounds of as many as fit the GPU, and a share costs about 64 keys' time besides its keys, so the
    // count that minimises rounds * (share + 64) - and never more pages per share than the kernel's table holds.
    const long long ctas = (long long)row_tiles * p.n_head_kv * p.st.n_seq;
    const int widest = GqaSmem(p.dim, p.out_dim, kMaxSharePages).bytes;
    if (widest > kSmemLimit) return launch_shared_kv_plain(p, INGOT_F16, s);
    const int slots = kv->num_sms * std::max(1, std::min(4, kSmemLimit / (GqaSmem(p.dim, p.out_dim, 64).bytes + 1024)));
    long long best = -1;
    for (int n = 1; n <= kMaxSplits; n++) {
        const int share = (pages * kBlockTokens + n - 1) / n;
        if (n > 1 && share < kSplitKeysMin) break;
        const long long cost = (ctas * n + slots - 1) / slots * (share + 64 + (n > 1 ? n : 0));
        if (best < 0 || cost < best) { best = cost; p.n_splits = n; }
    }
    p.n_splits = std::max(p.n_splits, (pages + kMaxSharePages - 1) / kMaxSharePages);
    if (p.n_splits > kMaxSplits) return launch_shared_kv_plain(p, INGOT_F16, s);
    const int share_pages = (pages + p.n_splits - 1) / p.n_splits, smem = GqaSmem(p.dim, p.out_dim, share_pages).bytes;
    if (p.n_splits > 1) {
        const size_t need = (size_t)p.st.n_tok * p.n_head * p.n_splits * (p.out_dim + 2);
        if (need > kv->part_floats) {
            float* fresh = nullptr;
            INGOT_CUDA_TRY(cudaMalloc(&fresh, need * sizeof(float)));
            if (kv->part) kv->retired.push_back(kv->part);  // a captured graph may still point into it
            kv->part = fresh;
            kv->part_floats = need;
        }
        p.part = kv->part;
    }
    const int most = std::max(p.q_dim, p.out_dim);
    auto kernel = most <= 64 ? gqa_mma_kernel<64> : most <= 128 ? gqa_mma_kernel<128> : gqa_mma_kernel<256>;
    INGOT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, widest));
    INGOT_CUDA_TRY(ingot_launch_pdl(kernel, dim3(row_tiles * p.n_splits, p.n_head_kv, p.st.n_seq), dim3(kWarps * 32), size_t(smem), s, p, share_pages));
    if (p.n_splits > 1) INGOT_CUDA_TRY(ingot_launch_pdl(gqa_merge_kernel, dim3(p.n_head, p.st.max_len, p.st.n_seq), dim3(128), 0, s, p));
    return INGOT_OK;
}

bool step_ok(const ingot_step* st) {
    return st && st->n_tok >= 1 && st->n_seq >= 1 && st->n_seq <= 65535 && st->max_len >= 1 && st->row_seq && st->row_start && st->len && st->pos0;
}
bool shape_ok(const ingot_skv* kv, const ingot_gqa_shape* sh) {
    return sh && sh->n_head >= 1 && sh->n_head_kv >= 1 && sh->n_head % sh->n_head_kv == 0 && sh->dim >= 4 && sh->dim % 4 == 0 && sh->vdim >= 4 && sh->vdim % 4 == 0 &&
           sh->dim_count >= 1 && sh->dim_count <= sh->dim && sh->rot_dims >= 0 && sh->rot_dims % 2 == 0 && sh->rot_dims <= sh->dim_count &&
           sh->norm >= INGOT_QK_NORM_NONE && sh->norm <= INGOT_QK_NORM_ALL && kv->n_head_kv == sh->n_head_kv && kv->dim == sh->dim + sh->vdim && !kv->inv_rms &&
           !kv->tiled && kv->chunk == 0;
}

}  // namespace

extern "C" {

int ingot_gqa_append(ingot_skv* kv, int layer, const ingot_step* step, const float* proj_dev, int proj_ld, int q_off, int k_off, int v_off,
                     const ingot_gqa_shape* shape, const float* q_norm_dev, const float* k_norm_dev, float eps, const double* turns_dev, float rot_gain,
                     float* first_values_dev, int store_first, float mix, void* q_out_dev, const int32_t* tables_dev, const int32_t* first_page_dev,
                     int max_blocks, void* stream) {
    INGOT_REQUIRE(kv && step_ok(step), "ingot_gqa_append: null handle or bad step");
    INGOT_REQUIRE_DEVICE(kv);
    INGOT_REQUIRE(layer >= 0 && layer < kv->n_layer, "ingot_gqa_append: layer out of range");
    INGOT_REQUIRE(shape_ok(kv, shape), "ingot_gqa_append: bad shape, or not a cache of joined rows of it");
    INGOT_REQUIRE(proj_dev && q_out_dev && tables_dev && max_blocks >= 1 && (turns_dev || shape->rot_dims == 0) &&
                      (shape->norm == INGOT_QK_NORM_NONE || (q_norm_dev && k_norm_dev)), "ingot_gqa_append: null argument");
    INGOT_REQUIRE(proj_ld % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0, "ingot_gqa_append: rows and offsets must be multiples of 4 floats");
    if (shape->rot_dims > kMaxRot) {
        ingot_set_error("ingot_gqa_append: at most " + std::to_string(kMaxRot) + " rotated values");
        return INGOT_ERR_UNSUPPORTED;
    }
    const size_t esz = kv->dtype == INGOT_F32 ? 4 : 2;
    AppendParams p = {*step, proj_dev, proj_ld, q_off, k_off, v_off, *shape, q_norm_dev, k_norm_dev, eps, turns_dev, rot_gain, first_values_dev, store_first, mix,
                      q_out_dev, static_cast<char*>(kv->rows) + kv->layer_elems * layer * esz, tables_dev, first_page_dev, max_blocks, kv->n_blocks, page_map(kv),
                      kv->status_dev};
    auto kernel = kv->dtype == INGOT_F32 ? gqa_append_kernel<float> : gqa_append_kernel<__half>;
    // few tokens: a CTA per eight heads, so that no warp has several in a row
    const int heads = shape->n_head + shape->n_head_kv, parts = step->n_tok <= 64 ? std::min(8, (heads + 7) / 8) : 1;
    INGOT_CUDA_TRY(ingot_launch_pdl(kernel, dim3(step->n_tok, parts), dim3(kAppendThreads), 0, static_cast<cudaStream_t>(stream), p));
    return INGOT_OK;
}

int ingot_gqa_attend(ingot_skv* kv, int layer, const ingot_step* step, const void* q_dev, const ingot_gqa_shape* shape, float scale, const float* sink_dev,
                     const float* gate_dev, int gate_ld, int gate_per_head, const ingot_act_out* out, const int32_t* tables_dev, const int32_t* first_page_dev,
                     int max_blocks, int impl, void* stream) {
    INGOT_REQUIRE(kv && step_ok(step), "ingot_gqa_attend: null handle or bad step");
    INGOT_REQUIRE_DEVICE(kv);
    INGOT_REQUIRE(layer >= 0 && layer < kv->n_layer, "ingot_gqa_attend: layer out of range");
    INGOT_REQUIRE(shape_ok(kv, shape), "ingot_gqa_attend: bad shape, or not a cache of joined rows of it");
    INGOT_REQUIRE(q_dev && out && tables_dev && max_blocks >= 1, "ingot_gqa_attend: null argument");
    INGOT_REQUIRE(out->ld % 2 == 0 && out->ld >= shape->n_head * shape->vdim && (!gate_dev || gate_ld % 4 == 0), "ingot_gqa_attend: bad output or gate rows");
    const size_t esz = kv->dtype == INGOT_F32 ? 4 : 2;
    AttendParams p = {*step, q_dev, static_cast<const char*>(kv->rows) + kv->layer_elems * layer * esz, nullptr, tables_dev, first_page_dev, max_blocks,
                      kv->n_blocks, shape->n_head, kv->n_head_kv, kv->dim, shape->vdim, page_map(kv), scale,
                      SharedOut{out->f32, static_cast<__nv_bfloat16*>(out->hi), static_cast<__nv_bfloat16*>(out->lo), out->ld, 1.0f}, kv->status_dev, 1, nullptr,
                      false, sink_dev, shape->dim, shape->dim, OutGate{gate_dev, gate_ld, gate_per_head}};
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (kv->dtype == INGOT_F16) {
        // The split-key kernel fills the GPU with any number of rows and reads the keys once per 16 of a KV head, the tcgen05 one walks them
        // in one CTA per 256: it wins when there are rows for many CTAs. INGOT_GQA_LONG sets the number.
        const char* env = getenv("INGOT_GQA_LONG");
        const long long least = env ? atoll(env) : INGOT_GQA_LONG_ROWS, rows = (long long)step->n_seq * step->max_len * shape->n_head;
        if ((impl == 3 || (impl == 0 && step->max_len > 1 && rows >= least)) && gqa_sm100_takes(shape->dim, shape->vdim, scale) && out->ld % 4 == 0) {
            const int rc = launch_gqa_sm100(kv, layer, p, s);
            if (rc != INGOT_ERR_UNSUPPORTED || impl == 3) return rc;
        }
        if ((impl == 0 || impl == 2) && mma_takes(shape->dim, shape->vdim)) return launch_mma(kv, p, s);
    }
    if (impl == 2 || impl == 3) {
        ingot_set_error("ingot_gqa_attend: the tensor-core kernel does not take this cache or these sizes");
        return INGOT_ERR_UNSUPPORTED;
    }
    return launch_shared_kv_plain(p, kv->dtype, s);
}

}  // extern "C"
