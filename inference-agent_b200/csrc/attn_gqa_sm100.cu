// Grouped-query attention over joined [key | value] rows for portions of prompts on the sm_100a tensor cores (attn_gqa.cu has the
// mechanism): the tcgen05 / TMA / tensor-memory pipeline of attn_shared_kv_sm100.cu with keys and values of unequal lengths, a window, a
// sink and an output gate.
//
// One CTA = one KV head x 256 rows (two 128-row tiles) of one sequence of the step, a row being a (token, head of the group) pair. It walks
// the pages its rows see in tiles of 128 keys = 8 pages. Operands come in units of 128 keys x 64 columns (16 KB, a TMA box of 16 x 64 per
// page): a key tile is ceil(dim / 64) units that start at column 0 of the rows, a value tile one or two that start at column dim. The last
// key unit reaches into the value; products stop at the key's last 16 columns. The last value unit is filled with zeros past the row.
// One ring of units serves both, in the order K0 | V0 K1 | V1 K2 | ..; a value tile of two units whose slots are not adjacent (the ring
// wraps) is multiplied unit by unit.
// Roles: warp 0 TMA, warp 1 MMA issue, warps 4-7 and 8-11 softmax of the two row tiles, one thread per row.
// Tensor memory: S0 S1 (128 columns each), O0 O1 (up to 128 each); P (f16) overwrites the first half of its S. MMA order:
//   QK(0,0) QK(1,0) | PV(0,j) QK(0,j+1) PV(1,j) QK(1,j+1) | ...
// Every mbarrier wait is bounded: on expiry all roles leave, copies in flight are drained, tensor memory is freed and the cache's
// status word gets its bit.
#include <mutex>

#include "attn_shared_kv.cuh"
#include "sm100_ptx.cuh"

namespace {

using namespace ingot_sm100;

constexpr int kTileRows = 128, kTileKeys = 128, kTilePages = kTileKeys / kBlockTokens, kUnit = 128 * 64 * 2, kPageUnit = kBlockTokens * 128;
constexpr int kAllUnits = 14;  // of shared memory: two query tiles and the ring
constexpr int kMaxRing = kAllUnits - 2;
constexpr int kThreads = 384;
constexpr uint32_t kTmemCols = 512;
constexpr float kRescaleThreshold = 8.0f;  // log2 units
constexpr unsigned long long kWaitLimitNs = 2000000000ull;
constexpr int kOffBar = kAllUnits * kUnit;
constexpr int kSmemBytes = kOffBar + 512 + 1024;  // + alignment slack

struct Bars {
    uint64_t full[kMaxRing];
    uint64_t empty[kMaxRing];
    uint64_t q_ready;
    uint64_t s_ready[2];
    uint64_t p_ready[2];
    uint64_t o_final[2];
    uint32_t tmem_base;
    uint32_t abort_flag;
};
static_assert(sizeof(Bars) <= 512, "barriers");

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float sigmoid(float z) { return __fdividef(1.0f, 1.0f + ex2(-1.44269504f * z)); }  // z -> -inf: 1 / inf
__device__ __forceinline__ void ffma2(float& d0, float& d1, float a0, float a1, float b, float c) {
    asm("{\n.reg .b64 ra, rb, rc, rd;\n"
        "mov.b64 ra, {%2, %3};\nmov.b64 rb, {%4, %4};\nmov.b64 rc, {%5, %5};\n"
        "fma.rn.f32x2 rd, ra, rb, rc;\nmov.b64 {%0, %1}, rd;\n}\n"
        : "=f"(d0), "=f"(d1) : "f"(a0), "f"(a1), "f"(b), "f"(c));
}
__device__ __forceinline__ void fadd2(float& d0, float& d1, float a0, float a1, float b0, float b1) {
    asm("{\n.reg .b64 ra, rb, rd;\n"
        "mov.b64 ra, {%2, %3};\nmov.b64 rb, {%4, %5};\n"
        "add.rn.f32x2 rd, ra, rb;\nmov.b64 {%0, %1}, rd;\n}\n"
        : "=f"(d0), "=f"(d1) : "f"(a0), "f"(a1), "f"(b0), "f"(b1));
}

// Instruction descriptors, kind::f16: f16 A and B, f32 accumulate, M = 128; scores: A and B K-major, N = 128; values: B MN-major
constexpr uint32_t kIdescQK = (1u << 4) | ((128u >> 3) << 17) | ((128u >> 4) << 24);
__device__ __forceinline__ uint32_t idesc_pv(int n) { return (1u << 4) | (1u << 16) | ((uint32_t)(n >> 3) << 17) | ((128u >> 4) << 24); }

__global__ void __launch_bounds__(kThreads, 1)
gqa_sm100_kernel(const __grid_constant__ CUtensorMap map_rows, const __grid_constant__ AttendParams p) {
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
    const int row_base = ((int)gridDim.x - 1 - (int)blockIdx.x) * 2 * kTileRows;  // later rows may see more keys, they go first
    if (row_base >= n_rows) {
        INGOT_PDL_WAIT();
        return;
    }
    const int last_row = min(row_base + 2 * kTileRows, n_rows) - 1;
    const int page_a = p.map.page(p.map.first_visible(pos0 + row_base / G)), page_b = p.map.page(pos0 + last_row / G);
    const int n_it = (page_b - page_a) / kTilePages + 1;
    const int nq = (p.q_dim + 63) / 64, nv = (p.out_dim + 63) / 64, k_steps = p.q_dim / 16, ring = kAllUnits - 2 * nq;
    const uint32_t ring_base = smem_base + 2 * nq * kUnit;

    if (threadIdx.x == 0) {
        for (int s = 0; s < ring; s++) { mbar_init(smem_u32(&bars->full[s]), 1); mbar_init(smem_u32(&bars->empty[s]), 1); }
        mbar_init(smem_u32(&bars->q_ready), 8);
        for (int q = 0; q < 2; q++) {
            mbar_init(smem_u32(&bars->s_ready[q]), 1);
            mbar_init(smem_u32(&bars->p_ready[q]), 4);
            mbar_init(smem_u32(&bars->o_final[q]), 1);
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
            int slot = 0, round = 0, armed = 0;
            bool ok = true;
            auto unit = [&](int x, int z) {  // columns x.. of this lane's page (block and head z)
                if (!ok) return;
                const uint32_t full = smem_u32(&bars->full[slot]);
                if (lane == 0) {
                    ok = mbar_wait(smem_u32(&bars->empty[slot]), (uint32_t)((round & 1) ^ 1), abort_flag, kWaitLimitNs);
                    if (ok) mbar_expect_tx(full, kUnit);
                }
                ok = __shfl_sync(0xffffffffu, ok, 0);
                if (!ok) return;
                if (lane < kTilePages) tma_load_3d(ring_base + slot * kUnit + lane * kPageUnit, &map_rows, x, 0, z, full);
                armed++;
                if (++slot == ring) { slot = 0; round++; }
            };
            int z = 0;
            for (int it = 0; it <= n_it && ok; it++) {
                if (it > 0)
                    for (int u = 0; u < nv; u++) unit(p.q_dim + u * 64, z);
                if (it < n_it) {
                    // pages past the last one, or without a valid block, are replaced by block 0: their keys are masked
                    const int page = page_a + it * kTilePages + lane;
                    int blk = 0;
                    if (lane < kTilePages && page <= page_b) blk = max(table_block(p.tables, p.first_page, p.max_blocks, p.n_blocks, seq, page, p.status), 0);
                    z = blk * p.n_head_kv + kvh;
                    for (int u = 0; u < nq; u++) unit(u * 64, z);
                }
            }
            if (!ok && lane == 0) {
                // copies already issued must land before the CTA's shared memory is released
                for (int i = max(0, armed - ring); i < armed; i++) {
                    const uint64_t t0 = globaltimer_ns();
                    while (!mbar_try_wait(smem_u32(&bars->full[i % ring]), (uint32_t)((i / ring) & 1)) && globaltimer_ns() - t0 < 100000000ull) {}
                }
            }
        } else if (warp_u == 1) {
            // ---------------- MMA issuer: the whole warp walks the loop, one elected lane issues ----------------
            int slot = 0, round = 0;  // of the next unit to be consumed
            bool ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(&bars->q_ready), 0, abort_flag, kWaitLimitNs)) != 0;
            auto wait_units = [&](int n) {  // the n units from the current place on have landed
                int s = slot, r = round;
                for (int u = 0; u < n && ok; u++) {
                    ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(&bars->full[s]), (uint32_t)(r & 1), abort_flag, kWaitLimitNs)) != 0;
                    if (++s == ring) { s = 0; r++; }
                }
            };
            auto advance = [&](int n) {
                slot += n;
                if (slot >= ring) { slot -= ring; round++; }
            };
            auto wrap = [&](int s) { return s >= ring ? s - ring : s; };
            auto issue_qk = [&](int q, int first) {
                for (int u = 0; u < nq; u++) {
                    const uint32_t a = smem_base + (q * nq + u) * kUnit, b = ring_base + wrap(first + u) * kUnit;
#pragma unroll
                    for (int ks = 0; ks < 4; ks++)
                        if (u * 4 + ks < k_steps)
                            tc_mma_ss(tmem + q * 128, make_desc(a + ks * 32, 16, 1024), make_desc(b + ks * 32, 16, 1024), kIdescQK, (u > 0 || ks > 0) ? 1u : 0u);
                }
                tc_commit(smem_u32(&bars->s_ready[q]));
            };
            auto issue_pv = [&](int q, int first, bool fresh) {
                const int step = first + nv <= ring ? nv : 1;  // units per instruction
                for (int u = 0; u < nv; u += step) {
                    const uint32_t v = ring_base + wrap(first + u) * kUnit;
#pragma unroll
                    for (int ks = 0; ks < 8; ks++)
                        tc_mma_ts(tmem + 256 + q * 128 + u * 64, tmem + q * 128 + ks * 8, make_desc(v + ks * 2048, kUnit, 1024), idesc_pv(step * 64),
                                  (!fresh || ks > 0) ? 1u : 0u);
                }
            };
            auto release = [&](int first, int n) {
                for (int u = 0; u < n; u++) tc_commit(smem_u32(&bars->empty[wrap(first + u)]));
            };
            wait_units(nq);
            if (ok) {
                tc_fence_after();
                if (elect_one()) {
                    issue_qk(0, slot);
                    issue_qk(1, slot);
                    release(slot, nq);
                }
                __syncwarp();
                advance(nq);
            }
            for (int j = 0; j < n_it && ok; j++) {
                const bool more = j + 1 < n_it;
                wait_units(more ? nv + nq : nv);
                if (!ok) break;
                const int v_slot = slot, k_slot = wrap(slot + nv);
#pragma unroll
                for (int q = 0; q < 2; q++) {
                    ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(&bars->p_ready[q]), (uint32_t)(j & 1), abort_flag, kWaitLimitNs)) != 0;
                    if (!ok) break;
                    tc_fence_after();
                    if (elect_one()) {
                        issue_pv(q, v_slot, j == 0);
                        if (q == 1) release(v_slot, nv);
                        if (more) {
                            issue_qk(q, k_slot);
                            if (q == 1) release(k_slot, nq);
                        } else {
                            tc_commit(smem_u32(&bars->o_final[q]));
                        }
                    }
                    __syncwarp();
                }
                advance(more ? nv + nq : nv);
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
            // Q rows into the tile's units (K-major, 128-byte swizzle), four rows per load instruction
            const int my_src = valid ? (int)((tok0 + tok) * p.n_head + head) : -1;
            const int piece = lane & 7, warp_row0 = (warp & 3) << 5;
            for (int u = 0; u < nq; u++) {
                unsigned char* qunit = smem_al + (q * nq + u) * kUnit;
                const int col = u * 64 + piece * 8;
                uint4 qv[8];
#pragma unroll
                for (int it = 0; it < 8; it++) {
                    const int src = __shfl_sync(0xffffffffu, my_src, it * 4 + (lane >> 3));
                    qv[it] = src >= 0 && col < p.q_dim ? *reinterpret_cast<const uint4*>(static_cast<const __half*>(p.q) + (size_t)src * p.q_dim + col) : make_uint4(0, 0, 0, 0);
                }
#pragma unroll
                for (int it = 0; it < 8; it++) {
                    const int r = warp_row0 + it * 4 + (lane >> 3);
                    *reinterpret_cast<uint4*>(qunit + r * 128 + ((piece ^ (r & 7)) << 4)) = qv[it];
                }
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&bars->q_ready));
        }
        float m_ref = 0.f, l = 0.f;
        bool ok = true;
        const float scale = p.scale * 1.44269504f;
        const int pos_min = __shfl_sync(0xffffffffu, pos, 0), vis_max = __shfl_sync(0xffffffffu, vis, 31);  // rows ascend with the lane
        for (int j = 0; j < n_it; j++) {
            ok = mbar_wait(smem_u32(&bars->s_ready[q]), (uint32_t)(j & 1), abort_flag, kWaitLimitNs);
            ok = __all_sync(0xffffffffu, ok) != 0;
            if (!ok) break;
            tc_fence_after();
            float s[128];
#pragma unroll
            for (int c = 0; c < 4; c++) tmem_ld32(s_tmem + c * 32, *reinterpret_cast<float(*)[32]>(&s[c * 32]));
            tmem_wait_ld();
            const int kp = page_a * kBlockTokens + j * kTileKeys;  // position of the tile's first key
            if (kp < vis_max || kp + kTileKeys - 1 > pos_min) {  // warp-uniform: some row of this warp needs the mask
                const int lo = vis - kp, hi = pos - kp;
#pragma unroll
                for (int i = 0; i < 128; i++)
                    if (i < lo || i > hi) s[i] = -INFINITY;
            }
            float mxa = fmaxf(s[0], s[1]), mxb = fmaxf(s[2], s[3]), mxc = fmaxf(s[4], s[5]), mxd = fmaxf(s[6], s[7]);
#pragma unroll
            for (int i = 8; i < 128; i += 8) {
                mxa = fmaxf(mxa, fmaxf(s[i], s[i + 1]));
                mxb = fmaxf(mxb, fmaxf(s[i + 2], s[i + 3]));
                mxc = fmaxf(mxc, fmaxf(s[i + 4], s[i + 5]));
                mxd = fmaxf(mxd, fmaxf(s[i + 6], s[i + 7]));
            }
            const float mx = fmaxf(fmaxf(mxa, mxb), fmaxf(mxc, mxd)) * scale;
            // Lazy rescale: the reference maximum moves only when the row's grew by more than 2^8. A row that has seen only masked
            // keys keeps -inf; its first finite maximum "grows" from there with a rescale factor of exactly 0.
            const bool grow = j == 0 || mx > m_ref + kRescaleThreshold;
            if (j == 0) {
                m_ref = mx;
            } else if (__any_sync(0xffffffffu, grow)) {
                const float alpha = grow ? ex2(m_ref - mx) : 1.0f;
                if (grow) { m_ref = mx; l *= alpha; }
                for (int c = 0; c < nv * 2; c++) {
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
                    ffma2(x0, x1, s[c * 64 + 2 * i], s[c * 64 + 2 * i + 1], scale, neg_m);
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
            if (lane == 0) mbar_arrive(smem_u32(&bars->p_ready[q]));
        }
        // ---------------- epilogue: O / l through the tile's Q buffer, row-contiguous stores ----------------
        const int my_row = valid ? (int)(tok0 + tok) : -1, warp_row0 = (warp & 3) << 5, piece = lane & 7;
        float4 gates[8];  // of the rows and columns this lane stores in a pass, requested ahead of the result
        auto load_gates = [&](int ps) {
            if (!p.gate.z) return;
            const int d = ps * 32 + piece * 4;
#pragma unroll
            for (int it = 0; it < 8; it++) {
                const int owner = it * 4 + (lane >> 3);
                const int row = __shfl_sync(0xffffffffu, my_row, owner), h = __shfl_sync(0xffffffffu, head, owner);
                if (row < 0 || d >= p.out_dim) continue;
                const float* z = p.gate.z + (size_t)row * p.gate.ld;
                gates[it] = p.gate.per_head ? make_float4(z[h], z[h], z[h], z[h]) : *reinterpret_cast<const float4*>(z + h * p.out_dim + d);
            }
        };
        load_gates(0);
        if (ok) {
            ok = mbar_wait(smem_u32(&bars->o_final[q]), 0, abort_flag, kWaitLimitNs);
            ok = __all_sync(0xffffffffu, ok) != 0;
        }
        if (ok) {
            tc_fence_after();
            float inv;
            if (p.sink) {
                const float sink = p.sink[head] * 1.44269504f, top = fmaxf(m_ref, sink), mine = exp2f(m_ref - top);
                inv = mine / (l * mine + exp2f(sink - top));
            } else {
                inv = 1.0f / l;
            }
            unsigned char* stage = smem_al + q * nq * kUnit;  // [128 rows][32 f32], 16-byte pieces XOR-swizzled by row
            for (int ps = 0; ps < 2 * nv && ps * 32 < p.out_dim; ps++) {
                if (ps) {
                    load_gates(ps);
                    __syncwarp();
                }
                unsigned char* my = stage + row_in_tile * 128;
                float o[32];
                tmem_ld32(o_tmem + ps * 32, o);
                tmem_wait_ld();
#pragma unroll
                for (int i = 0; i < 8; i++)
                    *reinterpret_cast<float4*>(my + ((i ^ (row_in_tile & 7)) << 4)) = make_float4(o[4 * i] * inv, o[4 * i + 1] * inv, o[4 * i + 2] * inv, o[4 * i + 3] * inv);
                __syncwarp();
                const int d = ps * 32 + piece * 4;
#pragma unroll
                for (int it = 0; it < 8; it++) {
                    const int owner = it * 4 + (lane >> 3);
                    const int row = __shfl_sync(0xffffffffu, my_row, owner), h = __shfl_sync(0xffffffffu, head, owner);
                    if (row < 0 || d >= p.out_dim) continue;
                    const int r = warp_row0 + owner;
                    float4 v = *reinterpret_cast<const float4*>(stage + r * 128 + ((piece ^ (r & 7)) << 4));
                    if (p.gate.z) { v.x *= sigmoid(gates[it].x); v.y *= sigmoid(gates[it].y); v.z *= sigmoid(gates[it].z); v.w *= sigmoid(gates[it].w); }
                    const size_t e = (size_t)row * p.out.ld + h * p.out_dim + d;  // out_dim is a multiple of 16
                    if (p.out.f32) *reinterpret_cast<float4*>(p.out.f32 + e) = v;
                    if (p.out.hi) {
                        const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
                        *reinterpret_cast<uint2*>(p.out.hi + e) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
                        if (p.out.lo) {
                            const __nv_bfloat162 c = __floats2bfloat162_rn(v.x - __low2float(a), v.y - __high2float(a)), f = __floats2bfloat162_rn(v.z - __low2float(b), v.w - __high2float(b));
                            *reinterpret_cast<uint2*>(p.out.lo + e) = make_uint2(*reinterpret_cast<const uint32_t*>(&c), *reinterpret_cast<const uint32_t*>(&f));
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

bool gqa_sm100_takes(int dim, int vdim, float scale) { return dim % 16 == 0 && vdim % 16 == 0 && dim <= 256 && vdim <= 128 && scale > 0; }

int launch_gqa_sm100(ingot_skv* kv, int layer, const AttendParams& p, cudaStream_t stream) {
    if (kv->dtype != INGOT_F16 || kv->tiled || kv->dim % 8 != 0) return INGOT_ERR_UNSUPPORTED;
    if (kv->tmaps.empty()) {
        EncodeTiledFn encode = encode_fn();
        if (!encode) return INGOT_ERR_UNSUPPORTED;
        std::vector<CUtensorMap> maps(kv->n_layer);
        for (int i = 0; i < kv->n_layer; i++) {
            const cuuint64_t dims[3] = {(cuuint64_t)kv->dim, kBlockTokens, (cuuint64_t)kv->n_blocks * kv->n_head_kv};
            const cuuint64_t strides[2] = {(cuuint64_t)kv->dim * 2, (cuuint64_t)kBlockTokens * kv->dim * 2};
            const cuuint32_t box[3] = {64, kBlockTokens, 1}, estr[3] = {1, 1, 1};
            if (encode(&maps[i], CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 3, static_cast<__half*>(kv->rows) + (size_t)i * kv->layer_elems, dims, strides, box, estr,
                       CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                       CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
                return INGOT_ERR_UNSUPPORTED;
        }
        INGOT_CUDA_TRY(cudaFuncSetAttribute(gqa_sm100_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemBytes));
        kv->tmaps = std::move(maps);
    }
    const int group = p.n_head / p.n_head_kv;
    const dim3 grid((unsigned)(((size_t)p.st.max_len * group + 2 * kTileRows - 1) / (2 * kTileRows)), p.n_head_kv, p.st.n_seq);
    INGOT_CUDA_TRY(ingot_launch_pdl(gqa_sm100_kernel, grid, dim3(kThreads), size_t(kSmemBytes), stream, kv->tmaps[layer], p));
    return INGOT_OK;
}
