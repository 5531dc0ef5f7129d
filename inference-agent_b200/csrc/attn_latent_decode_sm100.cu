// Latent attention of decoded tokens on the sm_100a tensor cores (attn_latent.cu has the mechanism). One token's heads are few and the
// cached rows long, so the products are turned round: keys, then latent columns, are the 128 rows of the MMAs, the heads their columns.
//     S^T [keys][heads]          = rows . q^T      A: the key tile as it lies in memory (K-major), B: the query rows
//     O^T [128 columns][heads] += rows^T . p^T     A: the same tile read along its other dimension (MN-major), B: the weights
// Nothing is padded but the heads (to 16 or 32), one tile of shared memory serves both products, and the whole result of 512 latent
// columns and 32 heads takes 128 columns of tensor memory. The kernel is bound by reading the rows.
//
// One CTA = up to 32 heads of one token x one share of its visible pages, in tiles of 64 keys = 4 pages, so that two tiles of the
// longest rows fit shared memory and one loads while the other is multiplied. Pages lie in memory as the MMAs want them (tiled order,
// page_elem): a page is one contiguous copy, the 8-key groups of a tile follow each other units * 1024 bytes apart, whatever the page.
// (The score MMAs still have 128 rows: the upper 64 read what follows the tile in shared memory and their results are not looked at.)
// Roles: warp 0 TMA, warp 1 MMA issue, warps 2-5 softmax. The scores come out of tensor memory with a key per thread, go through shared
// memory to a quarter of the heads per warp (two keys per lane), and back as f16 weights, the B operand of the second product.
// Every mbarrier wait is bounded: on expiry all roles leave, copies in flight are drained, tensor memory is freed and the cache's
// status word gets its bit.
#include <mutex>

#include "attn_shared_kv.cuh"
#include "sm100_ptx.cuh"

namespace {

using namespace ingot_sm100;

constexpr int kKeys = 64, kPages = kKeys / kBlockTokens;
constexpr int kThreads = 192;
constexpr int kMaxStages = 8;
constexpr float kRescaleThreshold = 8.0f;  // log2 units
constexpr unsigned long long kWaitLimitNs = 2000000000ull;
constexpr int kSmemLimit = 227 * 1024;

struct Bars {
    uint64_t full[kMaxStages];
    uint64_t empty[kMaxStages];
    uint64_t q_ready;
    uint64_t s_ready[2];
    uint64_t p_ready;
    uint64_t pv_done;
    uint32_t tmem_base;
    uint32_t abort_flag;
    uint32_t rescale;
};

template <int kN>  // heads per CTA
struct Layout {
    static constexpr int kP = kN * 128;         // weights [heads][64 keys]
    static constexpr int kS = kN * kKeys * 4;   // scores [heads][keys]
    int units, tile, stages, off_q, off_p, off_s, off_vec, off_bar, bytes;
    // The ring comes first, and the whole is at least a tile longer than it: the upper rows of the score MMAs stay inside.
    __host__ __device__ explicit Layout(int row) {
        units = row / 64;
        tile = kKeys * row * 2;
        const int fixed = units * kN * 128 + kP + kS + 2 * kN * 4 + int(sizeof(Bars)) + 64, limit = kSmemLimit - 1024;
        stages = 0;
        while (stages < kMaxStages && (stages + 1) * tile + fixed <= limit && (stages + 2) * tile <= limit) stages++;
        off_q = stages * tile;
        off_p = off_q + units * kN * 128;
        off_s = off_p + kP;
        off_vec = off_s + kS;
        off_bar = (off_vec + 2 * kN * 4 + 15) / 16 * 16;
        bytes = off_bar + int(sizeof(Bars));
        if (bytes < (stages + 1) * tile) bytes = (stages + 1) * tile;
        bytes += 1024;
    }
};

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// Barrier of the softmax warps; the second form says whether all of their threads passed true.
__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ bool softmax_all(bool v) {
    uint32_t r;
    asm volatile("{\n.reg .pred p, q;\nsetp.ne.u32 q, %1, 0;\nbar.red.and.pred p, 1, 128, q;\nselp.u32 %0, 1, 0, p;\n}\n" : "=r"(r) : "r"((uint32_t)v) : "memory");
    return r != 0;
}
template <int kN>
__device__ __forceinline__ void tmem_ld(uint32_t addr, float (&v)[kN]) {
    if constexpr (kN == 32) {
        tmem_ld32(addr, v);
    } else {
        uint32_t* r = reinterpret_cast<uint32_t*>(v);
        asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                     : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
                       "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
                     : "r"(addr) : "memory");
    }
}
template <int kN>
__device__ __forceinline__ void tmem_st(uint32_t addr, const uint32_t (&r)[kN]) {
    if constexpr (kN == 32) {
        tmem_st32(addr, r);
    } else {
        asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
                     ::"r"(addr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]),
                       "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
                     : "memory");
    }
}

// Instruction descriptors, kind::f16, f32 accumulate, M = 128: scores A and B K-major; values A MN-major, B K-major
template <int kN> constexpr uint32_t kIdescS = (1u << 4) | ((uint32_t)(kN >> 3) << 17) | ((128u >> 4) << 24);
template <int kN> constexpr uint32_t kIdescV = kIdescS<kN> | (1u << 15);

template <int kN>
__global__ void __launch_bounds__(kThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ AttendParams p) {
    constexpr int kHeadsPerWarp = kN / 4;
    extern __shared__ unsigned char smem_dyn[];
    INGOT_PDL_TRIGGER();
    const Layout<kN> L(p.dim);
    const uint32_t smem_base = (smem_u32(smem_dyn) + 1023u) & ~1023u;
    unsigned char* smem_al = smem_dyn + (smem_base - smem_u32(smem_dyn));
    Bars* bars = reinterpret_cast<Bars*>(smem_al + L.off_bar);
    volatile uint32_t* abort_flag = &bars->abort_flag;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int warp_u = __shfl_sync(0xffffffffu, warp, 0);

    const int seq = blockIdx.z, split = blockIdx.y, h0 = blockIdx.x * kN;
    const int pos = p.st.pos0[seq], vis = p.map.first_visible(pos);
    const size_t tok = p.st.row_start[seq];
    const int page_a = p.map.page(vis), page_b = p.map.page(pos);
    const int tiles = (page_b - page_a) / kPages + 1, per = (tiles + p.n_splits - 1) / p.n_splits;
    const int first = split * per, n_it = max(0, min(per, tiles - first)), page0 = page_a + first * kPages;
    const int units = L.units, stages = L.stages, blocks = (p.out_dim + 127) / 128;

    if (threadIdx.x == 0) {
        for (int s = 0; s < stages; s++) { mbar_init(smem_u32(&bars->full[s]), 1); mbar_init(smem_u32(&bars->empty[s]), 1); }
        mbar_init(smem_u32(&bars->q_ready), 1);
        mbar_init(smem_u32(&bars->s_ready[0]), 1);
        mbar_init(smem_u32(&bars->s_ready[1]), 1);
        mbar_init(smem_u32(&bars->p_ready), 4);
        mbar_init(smem_u32(&bars->pv_done), 1);
        bars->abort_flag = 0;
        bars->rescale = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    const uint32_t tmem_cols = (2 + blocks) * kN <= 64 ? 64 : (2 + blocks) * kN <= 128 ? 128 : (2 + blocks) * kN <= 256 ? 256 : 512;
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&bars->tmem_base)), "r"(tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    INGOT_PDL_WAIT();  // queries and the newest row come from the kernels before
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = bars->tmem_base;  // S0 S1 | O, one column per head each

    if (warp_u == 0) {
        // ---------------- producer: lanes 0-3 fetch one page each ----------------
        int armed = 0;
        bool ok = true;
        const uint32_t page_bytes = kBlockTokens * p.dim * 2;
        for (int it = 0; it < n_it; it++) {
            // pages past the last one, or without a valid block, are replaced by block 0: their keys are masked
            const int page = page0 + it * kPages + lane, s = it % stages;
            const int blk = lane < kPages && page <= page_b ? max(table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, page, p.status), 0) : 0;
            const uint32_t full = smem_u32(&bars->full[s]);
            if (lane == 0) {
                ok = mbar_wait(smem_u32(&bars->empty[s]), (uint32_t)(((it / stages) & 1) ^ 1), abort_flag, kWaitLimitNs);
                if (ok) mbar_expect_tx(full, L.tile);
            }
            ok = __shfl_sync(0xffffffffu, ok, 0);
            if (!ok) break;
            if (lane < kPages)
                bulk_load(smem_base + s * L.tile + lane * page_bytes, static_cast<const __half*>(p.rows) + (size_t)blk * kBlockTokens * p.dim, page_bytes, full);
            armed = it + 1;
            if (it == 0 && lane == 0) {
                mbar_expect_tx(smem_u32(&bars->q_ready), units * kN * 128);
                for (int u = 0; u < units; u++) tma_load_2d(smem_base + L.off_q + u * kN * 128, &map_q, u * 64, (int)tok * p.n_head + h0, smem_u32(&bars->q_ready));
            }
        }
        if (!ok && lane == 0) {
            // copies already issued must land before the CTA's shared memory is released
            for (int it = max(0, armed - stages); it < armed; it++) {
                const uint64_t t0 = globaltimer_ns();
                while (!mbar_try_wait(smem_u32(&bars->full[it % stages]), (uint32_t)((it / stages) & 1)) && globaltimer_ns() - t0 < 100000000ull) {}
            }
            const uint64_t t0 = globaltimer_ns();
            while (armed > 0 && !mbar_try_wait(smem_u32(&bars->q_ready), 0) && globaltimer_ns() - t0 < 100000000ull) {}
        }
    } else if (warp_u == 1) {
        // ---------------- MMA issuer: the whole warp walks the loop, one elected lane issues ----------------
        bool ok = n_it == 0 || __all_sync(0xffffffffu, mbar_wait(smem_u32(&bars->q_ready), 0, abort_flag, kWaitLimitNs)) != 0;
        const uint32_t group = units * 1024;  // bytes from one group of 8 keys to the next
        auto scores = [&](int it) {
            ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(&bars->full[it % stages]), (uint32_t)((it / stages) & 1), abort_flag, kWaitLimitNs)) != 0;
            if (!ok) return;
            tc_fence_after();
            if (elect_one()) {
                for (int u = 0; u < units; u++) {
                    const uint32_t a = smem_base + (it % stages) * L.tile + u * 1024, b = smem_base + L.off_q + u * kN * 128;
#pragma unroll
                    for (int ks = 0; ks < 4; ks++)
                        tc_mma_ss(tmem + (it & 1) * kN, make_desc(a + ks * 32, 16, group), make_desc(b + ks * 32, 16, 1024), kIdescS<kN>, (u > 0 || ks > 0) ? 1u : 0u);
                }
                tc_commit(smem_u32(&bars->s_ready[it & 1]));
            }
            __syncwarp();
        };
        if (n_it > 0 && ok) scores(0);
        for (int it = 0; it < n_it && ok; it++) {
            // The next tile's scores go first if it is there before this one's weights are - but this one is given back without
            // waiting for it, so that two tiles are on their way at a time.
            const bool more = it + 1 < n_it;
            bool ahead = false;
            for (int spin = 0; more && stages > 1 && ok && spin < (1 << 20); spin++) {
                if (__any_sync(0xffffffffu, mbar_test(smem_u32(&bars->p_ready), (uint32_t)(it & 1)))) break;
                if (__all_sync(0xffffffffu, mbar_test(smem_u32(&bars->full[(it + 1) % stages]), (uint32_t)(((it + 1) / stages) & 1)))) {
                    scores(it + 1);
                    ahead = true;
                    break;
                }
            }
            ok = ok && __all_sync(0xffffffffu, mbar_wait(smem_u32(&bars->p_ready), (uint32_t)(it & 1), abort_flag, kWaitLimitNs)) != 0;
            if (!ok) break;
            tc_fence_after();
            if (elect_one()) {
                for (int b = 0; b < blocks; b++) {
                    const uint32_t a = smem_base + (it % stages) * L.tile + b * 2048, w = smem_base + L.off_p;
#pragma unroll
                    for (int ks = 0; ks < kKeys / 16; ks++)
                        tc_mma_ss(tmem + (2 + b) * kN, make_desc(a + ks * 2 * group, 1024, group), make_desc(w + ks * 32, 16, 1024), kIdescV<kN>, (it > 0 || ks > 0) ? 1u : 0u);
                }
                tc_commit(smem_u32(&bars->empty[it % stages]));
                tc_commit(smem_u32(&bars->pv_done));
            }
            __syncwarp();
            if (more && !ahead) scores(it + 1);
        }
    } else {
        // ---------------- softmax warps ----------------
        const int quarter = warp & 3;  // of the tensor-memory lanes: this thread's key, later its latent columns
        const uint32_t lane_sel = (uint32_t)(quarter << 5) << 16;
        float* s_score = reinterpret_cast<float*>(smem_al + L.off_s);
        float* s_alpha = reinterpret_cast<float*>(smem_al + L.off_vec);  // [heads]; at the end: factors of the result
        volatile uint32_t* rescale = &bars->rescale;
        const float scale = p.scale * 1.44269504f;
        float m_ref[kHeadsPerWarp], l[kHeadsPerWarp];
#pragma unroll
        for (int h = 0; h < kHeadsPerWarp; h++) { m_ref[h] = -INFINITY; l[h] = 0.f; }
        bool ok = true;
        for (int it = 0; it < n_it; it++) {
            ok = mbar_wait(smem_u32(&bars->s_ready[it & 1]), (uint32_t)((it >> 1) & 1), abort_flag, kWaitLimitNs);
            ok = __all_sync(0xffffffffu, ok) != 0;
            if (ok && quarter < 2) {  // the tile's keys are the lower half of the lanes
                float s[kN];
                tc_fence_after();
                tmem_ld<kN>(tmem + (it & 1) * kN + lane_sel, s);
                tmem_wait_ld();
                const int key = quarter * 32 + lane, kp = (page0 + it * kPages) * kBlockTokens + key;
                const bool on = kp >= vis && kp <= pos;
#pragma unroll
                for (int h = 0; h < kN; h++) s_score[h * kKeys + key] = on ? s[h] * scale : -INFINITY;
            }
            ok = softmax_all(ok);
            if (!ok) break;  // all four warps together
            // this warp's heads, two keys per lane
            float2 v[kHeadsPerWarp];
            bool grows = false;
#pragma unroll
            for (int h = 0; h < kHeadsPerWarp; h++) {
                v[h] = *reinterpret_cast<const float2*>(s_score + (quarter * kHeadsPerWarp + h) * kKeys + lane * 2);
                grows = grows || fmaxf(v[h].x, v[h].y) > m_ref[h] + kRescaleThreshold;
            }
            // Lazy rescale: a head's reference maximum moves only when its maximum grew by more than 2^8 (always at the first tile,
            // every one of which holds a visible key).
            float alpha[kHeadsPerWarp];
#pragma unroll
            for (int h = 0; h < kHeadsPerWarp; h++) alpha[h] = 1.0f;
            if (__any_sync(0xffffffffu, grows)) {
#pragma unroll
                for (int h = 0; h < kHeadsPerWarp; h++) {
                    float mx = fmaxf(v[h].x, v[h].y);
#pragma unroll
                    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
                    if (mx > m_ref[h] + kRescaleThreshold) {
                        alpha[h] = ex2(m_ref[h] - mx);
                        l[h] *= alpha[h];
                        m_ref[h] = mx;
                    }
                }
                if (lane == 0 && it > 0) *rescale = 1;
            }
            if (it > 0 && lane == 0) {
#pragma unroll
                for (int h = 0; h < kHeadsPerWarp; h++) s_alpha[quarter * kHeadsPerWarp + h] = alpha[h];
            }
            if (it > 0) {  // the product before must be through with the weights' buffer, and with O if it is rescaled
                ok = mbar_wait(smem_u32(&bars->pv_done), (uint32_t)((it - 1) & 1), abort_flag, kWaitLimitNs);
                ok = __all_sync(0xffffffffu, ok) != 0;
            }
#pragma unroll
            for (int h = 0; h < kHeadsPerWarp; h++) {
                const float ref = m_ref[h] == -INFINITY ? 0.f : m_ref[h];
                const float p0 = ex2(v[h].x - ref), p1 = ex2(v[h].y - ref);
                l[h] += p0 + p1;
                const int head = quarter * kHeadsPerWarp + h;  // 16-byte pieces of its row XOR-swizzled
                *reinterpret_cast<uint32_t*>(smem_al + L.off_p + head * 128 + (((lane >> 2) ^ (head & 7)) << 4) + (lane & 3) * 4) = pack_half2_rn(p0, p1);
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            ok = softmax_all(ok);  // scores are read, factors and weights are in
            if (!ok) break;
            if (it > 0 && *rescale) {
                tc_fence_after();
                for (int b = 0; b < blocks; b++) {
                    float o[kN];
                    tmem_ld<kN>(tmem + (2 + b) * kN + lane_sel, o);
                    tmem_wait_ld();
                    uint32_t ob[kN];
#pragma unroll
                    for (int h = 0; h < kN; h++) ob[h] = __float_as_uint(o[h] * s_alpha[h]);
                    tmem_st<kN>(tmem + (2 + b) * kN + lane_sel, ob);
                }
                tmem_wait_st();
                softmax_sync();
                if (threadIdx.x == 64) *rescale = 0;
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&bars->p_ready));
        }
        // ---------------- epilogue ----------------
        if (ok && n_it > 0) {
            ok = mbar_wait(smem_u32(&bars->pv_done), (uint32_t)((n_it - 1) & 1), abort_flag, kWaitLimitNs);
            ok = __all_sync(0xffffffffu, ok) != 0;
        }
        float* s_max = s_alpha + kN;
#pragma unroll
        for (int h = 0; h < kHeadsPerWarp; h++) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) l[h] += __shfl_xor_sync(0xffffffffu, l[h], o);
            const int head = quarter * kHeadsPerWarp + h;
            if (lane == 0 && h0 + head < p.n_head) {
                if (p.n_splits == 1) {
                    float f = 1.0f, sum = l[h];
                    if (p.sink) {
                        const float sink = p.sink[h0 + head] * 1.44269504f, top = fmaxf(m_ref[h], sink);
                        f = exp2f(m_ref[h] - top);
                        sum = sum * f + exp2f(sink - top);
                    }
                    s_max[head] = f / sum;
                } else {
                    float* part = p.part + ((tok * p.n_head + h0 + head) * p.n_splits + split) * (p.out_dim + 2) + p.out_dim;
                    part[0] = m_ref[h];
                    part[1] = l[h];
                    s_max[head] = 1.0f;
                }
            }
        }
        softmax_sync();
        if (ok) {
            tc_fence_after();
            const int heads = min(kN, p.n_head - h0);
            for (int b = 0; b < blocks; b++) {
                float o[kN];
                if (n_it > 0) {
                    tmem_ld<kN>(tmem + (2 + b) * kN + lane_sel, o);
                    tmem_wait_ld();
                }
                const int d = b * 128 + quarter * 32 + lane;
                if (d >= p.out_dim) continue;
                if (p.n_splits == 1) {
#pragma unroll
                    for (int h = 0; h < kN; h++)
                        if (h < heads) p.out.store(tok, (h0 + h) * p.out_dim + d, o[h] * s_max[h]);
                } else {
                    float* part = p.part + ((tok * p.n_head + h0) * p.n_splits + split) * (p.out_dim + 2) + d;
                    const size_t next = (size_t)p.n_splits * (p.out_dim + 2);
#pragma unroll
                    for (int h = 0; h < kN; h++)
                        if (h < heads) part[h * next] = n_it > 0 ? o[h] : 0.f;
                }
            }
        }
    }
    // ---------------- teardown ----------------
    tc_fence_before();
    __syncthreads();
    if (threadIdx.x == 0 && *abort_flag) atomicOr(p.status, kDevErrBarrierTimeout);
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(tmem_cols) : "memory");
    }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeTiledFn encode_fn() {
    static EncodeTiledFn fn = nullptr;
    static std::once_flag once;
    std::call_once(once, [] {
        void* sym = nullptr;
        cudaDriverEntryPointQueryResult qres;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &qres) == cudaSuccess &&
            qres == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<EncodeTiledFn>(sym);
    });
    return fn;
}

}  // namespace

// Row lengths the kernel takes: whole units, the latent's blocks of 128 columns inside the row, at least one tile in shared memory.
bool latent_decode_takes(int row, int rank) {
    const int blocks = (rank + 127) / 128;
    return row % 64 == 0 && blocks * 128 <= row && blocks <= 4 && Layout<32>(row).stages >= 1 && encode_fn() != nullptr;
}
int latent_decode_heads(int n_head) { return n_head <= 16 ? 16 : 32; }

// Decoded tokens (every sequence of the step has one); n_splits and part are set. q_rows: rows of the query buffer.
int launch_latent_decode_sm100(const ingot_skv* kv, const AttendParams& p, cudaStream_t stream) {
    if (!kv->tiled) return INGOT_ERR_UNSUPPORTED;
    const int n = latent_decode_heads(p.n_head);
    CUtensorMap map_q;
    {
        const cuuint64_t dims[2] = {(cuuint64_t)kv->dim, (cuuint64_t)p.st.n_tok * p.n_head};
        const cuuint64_t strides[1] = {(cuuint64_t)kv->dim * 2};
        const cuuint32_t box[2] = {64, (cuuint32_t)n}, estr[2] = {1, 1};
        if (encode_fn()(&map_q, CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 2, const_cast<void*>(p.q), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
            return INGOT_ERR_UNSUPPORTED;
    }
    const dim3 grid((p.n_head + n - 1) / n, p.n_splits, p.st.n_seq);
    if (n == 16) {
        const int smem = Layout<16>(kv->dim).bytes;
        INGOT_CUDA_TRY(cudaFuncSetAttribute(latent_decode_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        INGOT_CUDA_TRY(ingot_launch_pdl(latent_decode_kernel<16>, grid, dim3(kThreads), size_t(smem), stream, map_q, p));
    } else {
        const int smem = Layout<32>(kv->dim).bytes;
        INGOT_CUDA_TRY(cudaFuncSetAttribute(latent_decode_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        INGOT_CUDA_TRY(ingot_launch_pdl(latent_decode_kernel<32>, grid, dim3(kThreads), size_t(smem), stream, map_q, p));
    }
    return INGOT_OK;
}
