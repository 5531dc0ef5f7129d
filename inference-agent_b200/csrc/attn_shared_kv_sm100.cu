// Shared-row attention for portions of prompts on the sm_100a tensor cores: the tcgen05 / TMA / tensor-memory pipeline of
// attn_prefill_sm100.cu for caches whose rows are key and value at once (attn_shared_kv.cu has the mechanism), rows of 128
// f16 values.
//
// One CTA = one KV head x 256 rows (two 128-row tiles) of one sequence of the step, a row being a (token, head of the group)
// pair. It walks the visible keys in tiles of 128 = 8 pages. What differs from the K + V kernel:
//   - one TMA tile per step instead of two: the tile is the K-major B operand of S = Q K^T and, unchanged, the MN-major B
//     operand of O += P V, so the four 32 KB slots of the ring reach four steps ahead and half the bytes move;
//   - a key's scale (1/rms * score scale * log2 e) and position travel with the tile: warp 2 fetches them into arrays beside the
//     ring, and the softmax warps multiply every score by its key's scale;
//   - rows of one tile may belong to different chunks, so masks compare key positions with each row's first and last visible one.
// Roles: warp 0 TMA, warp 1 MMA issue, warp 2 scales, warps 4-7 and 8-11 softmax of the two row tiles, one thread per row.
// Tensor memory: S0 S1 O0 O1, 128 columns each; P (f16) overwrites the first half of its S. MMA order, as in the other kernel:
//   QK(0,0) QK(1,0) | PV(0,j) QK(0,j+1) PV(1,j) QK(1,j+1) | ...
// Every mbarrier wait is bounded: on expiry all roles leave, copies in flight are drained, tensor memory is freed and the
// cache's status word gets its bit.
#include "attn_shared_kv.cuh"
#include "sm100_ptx.cuh"

#include <mutex>

namespace {

using namespace ingot_sm100;

constexpr int kDim = 128, kTileRows = 128, kTileKeys = 128, kTilePages = kTileKeys / kBlockTokens;
constexpr int kStages = 4, kStageBytes = kTileKeys * kDim * 2, kHalfBytes = kStageBytes / 2, kQBytes = kTileRows * kDim * 2;
constexpr int kThreads = 384;
constexpr uint32_t kTmemCols = 512;
constexpr float kRescaleThreshold = 8.0f;  // log2 units
constexpr unsigned long long kWaitLimitNs = 2000000000ull;
constexpr int kNoKey = 0x7fffffff;

constexpr int kOffRing = 2 * kQBytes;
constexpr int kOffScale = kOffRing + kStages * kStageBytes;       // f32 [slot][128]
constexpr int kOffPos = kOffScale + kStages * kTileKeys * 4;      // int32 [slot][128]
constexpr int kOffBar = kOffPos + kStages * kTileKeys * 4;
constexpr int kSmemBytes = kOffBar + 256 + 1024;                  // + alignment slack

struct Bars {
    uint64_t full[kStages];   // two arrivals: the TMA producer (with the byte count) and the scale warp
    uint64_t empty[kStages];
    uint64_t q_ready;
    uint64_t s_ready[2];
    uint64_t p_ready[2];
    uint64_t o_final[2];
    int last_pos[kStages];    // largest key position of the slot (kNoKey if a key of it does not exist)
    uint32_t tmem_base;
    uint32_t abort_flag;
};

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void fmul2(float& d0, float& d1, float a0, float a1, float b0, float b1) {
    asm("{\n.reg .b64 ra, rb, rd;\n"
        "mov.b64 ra, {%2, %3};\nmov.b64 rb, {%4, %5};\n"
        "mul.rn.f32x2 rd, ra, rb;\nmov.b64 {%0, %1}, rd;\n}\n"
        : "=f"(d0), "=f"(d1) : "f"(a0), "f"(a1), "f"(b0), "f"(b1));
}
__device__ __forceinline__ void fadd2(float& d0, float& d1, float a0, float a1, float b0, float b1) {
    asm("{\n.reg .b64 ra, rb, rd;\n"
        "mov.b64 ra, {%2, %3};\nmov.b64 rb, {%4, %5};\n"
        "add.rn.f32x2 rd, ra, rb;\nmov.b64 {%0, %1}, rd;\n}\n"
        : "=f"(d0), "=f"(d1) : "f"(a0), "f"(a1), "f"(b0), "f"(b1));
}

// Instruction descriptor, kind::f16: f16 A and B, f32 accumulate, M = 128, N = 128.
constexpr uint32_t kIdescQK = (1u << 4) | ((128u >> 3) << 17) | ((128u >> 4) << 24);  // A and B K-major
constexpr uint32_t kIdescPV = kIdescQK | (1u << 16);                                    // B (the same tile as V) MN-major

__global__ void __launch_bounds__(kThreads, 1)
shared_kv_sm100_kernel(const __grid_constant__ CUtensorMap map_rows, const __grid_constant__ AttendParams p) {
    extern __shared__ unsigned char smem_dyn[];
    INGOT_PDL_TRIGGER();
    const uint32_t smem_base = (smem_u32(smem_dyn) + 1023u) & ~1023u;
    unsigned char* smem_al = smem_dyn + (smem_base - smem_u32(smem_dyn));
    Bars* bars = reinterpret_cast<Bars*>(smem_al + kOffBar);
    volatile uint32_t* abort_flag = &bars->abort_flag;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int warp_u = __shfl_sync(0xffffffffu, warp, 0);

    const int seq = blockIdx.z, kvh = blockIdx.y, G = p.n_head / p.n_head_kv;
    const int pos0 = p.st.pos0[seq], n_rows = p.st.len[seq] * G;
    const size_t tok0 = p.st.row_start[seq];
    const int row_base = ((int)gridDim.x - 1 - (int)blockIdx.x) * 2 * kTileRows;  // later rows see more keys, they go first
    if (row_base >= n_rows) {
        INGOT_PDL_WAIT();
        return;
    }
    const int last_row = min(row_base + 2 * kTileRows, n_rows) - 1;
    const int page_a = p.map.page(p.map.first_visible(pos0 + row_base / G)), page_b = p.map.page(pos0 + last_row / G);
    const int n_it = (page_b - page_a) / kTilePages + 1;  // at least one

    auto bar_addr = [&](const uint64_t* b) { return smem_u32(b); };
    if (threadIdx.x == 0) {
        for (int s = 0; s < kStages; s++) { mbar_init(bar_addr(&bars->full[s]), 2); mbar_init(bar_addr(&bars->empty[s]), 1); }
        mbar_init(bar_addr(&bars->q_ready), 8);
        for (int q = 0; q < 2; q++) {
            mbar_init(bar_addr(&bars->s_ready[q]), 1);
            mbar_init(bar_addr(&bars->p_ready[q]), 4);
            mbar_init(bar_addr(&bars->o_final[q]), 1);
        }
        bars->abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&bars->tmem_base)), "r"(kTmemCols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    INGOT_PDL_WAIT();  // q and the newest rows come from the kernel before
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = bars->tmem_base;

    if (warp_u < 4) {
        asm volatile("setmaxnreg.dec.sync.aligned.u32 56;");
        if (warp_u == 0) {
            // ---------------- TMA producer: lanes 0-7 fetch one page each ----------------
            int armed = 0;
            bool ok = true;
            for (int it = 0; it < n_it; it++) {
                const int s = it % kStages;
                const uint32_t full = bar_addr(&bars->full[s]);
                if (lane == 0) {
                    ok = mbar_wait(bar_addr(&bars->empty[s]), (uint32_t)(((it / kStages) & 1) ^ 1), abort_flag, kWaitLimitNs);
                    if (ok) mbar_expect_tx(full, kStageBytes);
                }
                ok = __shfl_sync(0xffffffffu, ok, 0);
                if (!ok) break;
                if (lane < kTilePages) {
                    // pages past the last one, or without a valid block, are replaced by block 0: their keys are masked
                    const int page = page_a + it * kTilePages + lane;
                    const int blk = page <= page_b ? max(table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, page, p.status), 0) : 0;
                    const uint32_t dst = smem_base + kOffRing + s * kStageBytes + lane * (kBlockTokens * 128);
                    const int z = blk * p.n_head_kv + kvh;
                    tma_load_3d(dst, &map_rows, 0, 0, z, full);
                    tma_load_3d(dst + kHalfBytes, &map_rows, 64, 0, z, full);
                }
                armed = it + 1;
            }
            if (!ok && lane == 0) {
                // copies already issued must land before the CTA's shared memory is released
                for (int it = max(0, armed - kStages); it < armed; it++) {
                    const uint64_t t0 = globaltimer_ns();
                    while (!mbar_try_wait(bar_addr(&bars->full[it % kStages]), (uint32_t)((it / kStages) & 1)) && globaltimer_ns() - t0 < 100000000ull) {}
                }
            }
        } else if (warp_u == 2) {
            // ---------------- scales and positions: four keys per lane ----------------
            float* s_scale = reinterpret_cast<float*>(smem_al + kOffScale);
            int* s_pos = reinterpret_cast<int*>(smem_al + kOffPos);
            for (int it = 0; it < n_it; it++) {
                const int s = it % kStages, page = page_a + it * kTilePages + (lane >> 2), slot0 = (lane & 3) * 4;
                const int blk = page <= page_b ? table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, page, p.status) : -1;
                float4 sc = make_float4(0.f, 0.f, 0.f, 0.f);
                int4 kp = make_int4(kNoKey, kNoKey, kNoKey, kNoKey);
                if (blk >= 0) {
                    sc = *reinterpret_cast<const float4*>(p.inv_rms + (size_t)blk * kBlockTokens + slot0);
                    const float f = p.scale * 1.44269504f;
                    sc.x *= f; sc.y *= f; sc.z *= f; sc.w *= f;
                    const int c = p.map.chunk > 0 ? page / p.map.pages_per_chunk : 0;
                    const int rel = (page - c * p.map.pages_per_chunk) * kBlockTokens + slot0, base = c * p.map.chunk + rel;
                    const int left = p.map.chunk > 0 ? p.map.chunk - rel : 4;  // keys of the chunk from here on
                    if (left > 0) kp.x = base;
                    if (left > 1) kp.y = base + 1;
                    if (left > 2) kp.z = base + 2;
                    if (left > 3) kp.w = base + 3;
                }
                bool ok = mbar_wait(bar_addr(&bars->empty[s]), (uint32_t)(((it / kStages) & 1) ^ 1), abort_flag, kWaitLimitNs);
                ok = __all_sync(0xffffffffu, ok) != 0;
                if (!ok) break;
                *reinterpret_cast<float4*>(s_scale + s * kTileKeys + lane * 4) = sc;
                *reinterpret_cast<int4*>(s_pos + s * kTileKeys + lane * 4) = kp;
                const int top = __reduce_max_sync(0xffffffffu, max(max(kp.x, kp.y), max(kp.z, kp.w)));
                if (lane == 0) bars->last_pos[s] = top;
                __syncwarp();
                if (lane == 0) mbar_arrive(bar_addr(&bars->full[s]));
            }
        } else if (warp_u == 1) {
            // ---------------- MMA issuer: the whole warp walks the loop, one elected lane issues ----------------
            const uint32_t q_base = smem_base;
            auto tile_addr = [&](int it) { return smem_base + kOffRing + (it % kStages) * kStageBytes; };
            auto wait_full = [&](int it) {
                return __all_sync(0xffffffffu, mbar_wait(bar_addr(&bars->full[it % kStages]), (uint32_t)((it / kStages) & 1), abort_flag, kWaitLimitNs)) != 0;
            };
            auto issue_qk = [&](int q, uint32_t k_addr) {
#pragma unroll
                for (int ks = 0; ks < 8; ks++) {
                    const uint32_t off = (ks >> 2) * kHalfBytes + (ks & 3) * 32;
                    tc_mma_ss(tmem + q * 128, make_desc(q_base + q * kQBytes + off, 16, 1024), make_desc(k_addr + off, 16, 1024), kIdescQK, ks > 0);
                }
                tc_commit(bar_addr(&bars->s_ready[q]));
            };
            auto issue_pv = [&](int q, uint32_t v_addr, bool first) {
#pragma unroll
                for (int ks = 0; ks < 8; ks++)
                    tc_mma_ts(tmem + 256 + q * 128, tmem + q * 128 + ks * 8, make_desc(v_addr + ks * 2048, kHalfBytes, 1024), kIdescPV,
                              (!first || ks > 0) ? 1u : 0u);
            };
            bool ok = __all_sync(0xffffffffu, mbar_wait(bar_addr(&bars->q_ready), 0, abort_flag, kWaitLimitNs)) != 0;
            ok = ok && wait_full(0);
            if (ok) {
                tc_fence_after();
                if (elect_one()) {
                    issue_qk(0, tile_addr(0));
                    issue_qk(1, tile_addr(0));
                }
                __syncwarp();
            }
            for (int j = 0; j < n_it && ok; j++) {
                const bool more = j + 1 < n_it;
                ok = !more || wait_full(j + 1);
                if (!ok) break;
                const uint32_t v_addr = tile_addr(j), k_addr = tile_addr(j + 1);
#pragma unroll
                for (int q = 0; q < 2; q++) {
                    ok = __all_sync(0xffffffffu, mbar_wait(bar_addr(&bars->p_ready[q]), (uint32_t)(j & 1), abort_flag, kWaitLimitNs)) != 0;
                    if (!ok) break;
                    tc_fence_after();
                    if (elect_one()) {
                        issue_pv(q, v_addr, j == 0);
                        if (q == 1) tc_commit(bar_addr(&bars->empty[j % kStages]));  // both tiles are done with slot j
                        if (more) issue_qk(q, k_addr);
                        else tc_commit(bar_addr(&bars->o_final[q]));
                    }
                    __syncwarp();
                }
            }
        }
    } else {
        asm volatile("setmaxnreg.inc.sync.aligned.u32 224;");
        // ---------------- softmax warps: one thread per row ----------------
        const int q = (warp - 4) >> 2, row_in_tile = ((warp & 3) << 5) | lane;
        const int R = row_base + q * kTileRows + row_in_tile;
        const bool valid = R < n_rows;
        const int Rc = valid ? R : n_rows - 1;  // rows past the end behave like the last row
        const int tok = Rc / G, head = kvh * G + Rc % G;
        const int pos = pos0 + tok, vis = p.map.first_visible(pos);
        const uint32_t lane_sel = (uint32_t)((warp & 3) << 5) << 16;
        const uint32_t s_tmem = tmem + q * 128 + lane_sel, o_tmem = tmem + 256 + q * 128 + lane_sel;
        {
            // Q rows into the tile's buffer (K-major, 128-byte swizzle), two rows per load instruction, all loads first
            const int my_src = valid ? (int)((tok0 + tok) * p.n_head + head) : -1;
            unsigned char* qtile = smem_al + q * kQBytes;
            const int piece = lane & 15, warp_row0 = (warp & 3) << 5;
            uint4 qv[16];
#pragma unroll
            for (int it = 0; it < 16; it++) {
                const int src = __shfl_sync(0xffffffffu, my_src, it * 2 + (lane >> 4));
                qv[it] = src >= 0 ? *reinterpret_cast<const uint4*>(static_cast<const __half*>(p.q) + (size_t)src * kDim + piece * 8) : make_uint4(0, 0, 0, 0);
            }
#pragma unroll
            for (int it = 0; it < 16; it++) {
                const int r = warp_row0 + it * 2 + (lane >> 4);
                *reinterpret_cast<uint4*>(qtile + (piece >> 3) * kHalfBytes + r * 128 + (((piece & 7) ^ (r & 7)) << 4)) = qv[it];
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_addr(&bars->q_ready));
        }
        float m_ref = 0.f, l = 0.f;
        bool ok = true;
        const int pos_min = __shfl_sync(0xffffffffu, pos, 0), vis_max = __shfl_sync(0xffffffffu, vis, 31);  // rows ascend with the lane
        for (int j = 0; j < n_it; j++) {
            const int slot = j % kStages;
            ok = mbar_wait(bar_addr(&bars->s_ready[q]), (uint32_t)(j & 1), abort_flag, kWaitLimitNs);
            // the slot's barrier completed before its scores were computed: this only orders the scale warp's stores
            ok = ok && mbar_wait(bar_addr(&bars->full[slot]), (uint32_t)((j / kStages) & 1), abort_flag, kWaitLimitNs);
            ok = __all_sync(0xffffffffu, ok) != 0;
            if (!ok) break;
            tc_fence_after();
            float s[128];
#pragma unroll
            for (int c = 0; c < 4; c++) tmem_ld32(s_tmem + c * 32, *reinterpret_cast<float(*)[32]>(&s[c * 32]));
            tmem_wait_ld();
            const float4* ks = reinterpret_cast<const float4*>(smem_al + kOffScale) + slot * (kTileKeys / 4);
#pragma unroll
            for (int i = 0; i < 32; i++) {
                const float4 k = ks[i];
                fmul2(s[4 * i], s[4 * i + 1], s[4 * i], s[4 * i + 1], k.x, k.y);
                fmul2(s[4 * i + 2], s[4 * i + 3], s[4 * i + 2], s[4 * i + 3], k.z, k.w);
            }
            const int4* kp = reinterpret_cast<const int4*>(smem_al + kOffPos) + slot * (kTileKeys / 4);
            if (kp[0].x < vis_max || bars->last_pos[slot] > pos_min) {  // warp-uniform: some row of this warp needs the mask
#pragma unroll
                for (int i = 0; i < 32; i++) {
                    const int4 k = kp[i];
                    if (k.x < vis || k.x > pos) s[4 * i] = -INFINITY;
                    if (k.y < vis || k.y > pos) s[4 * i + 1] = -INFINITY;
                    if (k.z < vis || k.z > pos) s[4 * i + 2] = -INFINITY;
                    if (k.w < vis || k.w > pos) s[4 * i + 3] = -INFINITY;
                }
            }
            float mxa = fmaxf(s[0], s[1]), mxb = fmaxf(s[2], s[3]), mxc = fmaxf(s[4], s[5]), mxd = fmaxf(s[6], s[7]);
#pragma unroll
            for (int i = 8; i < 128; i += 8) {
                mxa = fmaxf(mxa, fmaxf(s[i], s[i + 1]));
                mxb = fmaxf(mxb, fmaxf(s[i + 2], s[i + 3]));
                mxc = fmaxf(mxc, fmaxf(s[i + 4], s[i + 5]));
                mxd = fmaxf(mxd, fmaxf(s[i + 6], s[i + 7]));
            }
            const float mx = fmaxf(fmaxf(mxa, mxb), fmaxf(mxc, mxd));
            // Lazy rescale: the reference maximum moves only when the row's grew by more than 2^8. A row that has seen only masked
            // keys keeps -inf; its first finite maximum "grows" from there with a rescale factor of exactly 0.
            const bool grow = j == 0 || mx > m_ref + kRescaleThreshold;
            if (j == 0) {
                m_ref = mx;
            } else if (__any_sync(0xffffffffu, grow)) {
                const float alpha = grow ? ex2(m_ref - mx) : 1.0f;
                if (grow) { m_ref = mx; l *= alpha; }
#pragma unroll
                for (int c = 0; c < 4; c++) {
                    float o[32];
                    tmem_ld32(o_tmem + c * 32, o);
                    tmem_wait_ld();
                    uint32_t ob[32];
#pragma unroll
                    for (int i = 0; i < 32; i++) ob[i] = __float_as_uint(o[i] * alpha);
                    tmem_st32(o_tmem + c * 32, ob);
                }
            }
            const float neg_m = m_ref == -INFINITY ? 0.f : -m_ref;
            float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
            for (int c = 0; c < 2; c++) {
                uint32_t pk[32];
#pragma unroll
                for (int i = 0; i < 32; i++) {
                    float x0, x1;
                    fadd2(x0, x1, s[c * 64 + 2 * i], s[c * 64 + 2 * i + 1], neg_m, neg_m);
                    const float p0 = ex2(x0), p1 = ex2(x1);
                    fadd2(sum0, sum1, sum0, sum1, p0, p1);
                    pk[i] = pack_half2_rn(p0, p1);
                }
                tmem_st32(s_tmem + c * 32, pk);
            }
            l += sum0 + sum1;
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_addr(&bars->p_ready[q]));
        }
        // ---------------- epilogue: O / l through the tile's Q buffer, row-contiguous stores ----------------
        if (ok) {
            ok = mbar_wait(bar_addr(&bars->o_final[q]), 0, abort_flag, kWaitLimitNs);
            ok = __all_sync(0xffffffffu, ok) != 0;
        }
        if (ok) {
            tc_fence_after();
            const float inv = p.out.scale / l;
            unsigned char* stage = smem_al + q * kQBytes;  // [128 rows][64 f32], 16-byte pieces XOR-swizzled by row
            const int my_row = valid ? (int)(tok0 + tok) : -1, warp_row0 = (warp & 3) << 5, piece = lane & 15;
            for (int ps = 0; ps < 2; ps++) {
                if (ps) __syncwarp();
                unsigned char* my = stage + row_in_tile * 256;
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    float o[32];
                    tmem_ld32(o_tmem + ps * 64 + c * 32, o);
                    tmem_wait_ld();
#pragma unroll
                    for (int i = 0; i < 8; i++)
                        *reinterpret_cast<float4*>(my + (((c * 8 + i) ^ (row_in_tile & 7)) << 4)) =
                            make_float4(o[4 * i] * inv, o[4 * i + 1] * inv, o[4 * i + 2] * inv, o[4 * i + 3] * inv);
                }
                __syncwarp();
                const int d = ps * 64 + piece * 4;
#pragma unroll 4
                for (int it = 0; it < 16; it++) {
                    const int owner = it * 2 + (lane >> 4);
                    const int row = __shfl_sync(0xffffffffu, my_row, owner), h = __shfl_sync(0xffffffffu, head, owner);
                    if (row < 0 || d >= p.out_dim) continue;
                    const int r = warp_row0 + owner;
                    const float4 v = *reinterpret_cast<const float4*>(stage + r * 256 + ((piece ^ (r & 7)) << 4));
                    const size_t e = (size_t)row * p.out.ld + h * p.out_dim + d;
                    if (p.out_dim % 4 == 0 && p.out.ld % 4 == 0) {
                        if (p.out.f32) *reinterpret_cast<float4*>(p.out.f32 + e) = v;
                        if (p.out.hi) {
                            const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
                            *reinterpret_cast<uint2*>(p.out.hi + e) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
                            if (p.out.lo) {
                                const float2 af = __bfloat1622float2(a), bf = __bfloat1622float2(b);
                                const __nv_bfloat162 c = __floats2bfloat162_rn(v.x - af.x, v.y - af.y), f = __floats2bfloat162_rn(v.z - bf.x, v.w - bf.y);
                                *reinterpret_cast<uint2*>(p.out.lo + e) = make_uint2(*reinterpret_cast<const uint32_t*>(&c), *reinterpret_cast<const uint32_t*>(&f));
                            }
                        }
                    } else {
                        const float f[4] = {v.x, v.y, v.z, v.w};
                        for (int i = 0; i < 4 && d + i < p.out_dim; i++) {
                            if (p.out.f32) p.out.f32[e + i] = f[i];
                            if (p.out.hi) {
                                const __nv_bfloat16 hv = __float2bfloat16_rn(f[i]);
                                p.out.hi[e + i] = hv;
                                if (p.out.lo) p.out.lo[e + i] = __float2bfloat16_rn(f[i] - __bfloat162float(hv));
                            }
                        }
                    }
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
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kTmemCols) : "memory");
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

int launch_shared_kv_sm100(ingot_skv* kv, int layer, const AttendParams& p, cudaStream_t stream) {
    if (kv->dim != kDim || kv->dtype != INGOT_F16) return INGOT_ERR_UNSUPPORTED;
    if (kv->tmaps.empty()) {
        EncodeTiledFn encode = encode_fn();
        if (!encode) return INGOT_ERR_UNSUPPORTED;
        std::vector<CUtensorMap> maps(kv->n_layer);
        for (int i = 0; i < kv->n_layer; i++) {
            const cuuint64_t dims[3] = {kDim, kBlockTokens, (cuuint64_t)kv->n_blocks * kv->n_head_kv};
            const cuuint64_t strides[2] = {kDim * 2, kBlockTokens * kDim * 2};
            const cuuint32_t box[3] = {64, kBlockTokens, 1}, estr[3] = {1, 1, 1};
            if (encode(&maps[i], CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 3, static_cast<__half*>(kv->rows) + (size_t)i * kv->layer_elems, dims, strides, box, estr,
                       CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                       CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
                return INGOT_ERR_UNSUPPORTED;
        }
        INGOT_CUDA_TRY(cudaFuncSetAttribute(shared_kv_sm100_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemBytes));
        kv->tmaps = std::move(maps);
    }
    const int group = p.n_head / p.n_head_kv;
    const dim3 grid((unsigned)(((size_t)p.st.max_len * group + 2 * kTileRows - 1) / (2 * kTileRows)), p.n_head_kv, p.st.n_seq);
    INGOT_CUDA_TRY(ingot_launch_pdl(shared_kv_sm100_kernel, grid, dim3(kThreads), size_t(kSmemBytes), stream, kv->tmaps[layer], p));
    return INGOT_OK;
}
