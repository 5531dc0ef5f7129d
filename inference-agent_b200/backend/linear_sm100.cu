// Batched projections of CudaBackend::forward_batch on the sm_100a tensor cores:
//   out[t][r] (+)= sum_i W[r][i] * x[t][i]      W f16 [n_out][n_in] (ggml ne = [n_in, n_out]), x and out f32
// — the job of the matmul loops of the CPU reference (src/cpu_backend.cpp:39-42, 71-85 over
// ops::dot_row, src/ops.cpp:127-141) and of Metal's matmul_f16 (src/metal_backend.mm:282-322) for a
// prefill chunk of up to n_batch tokens.
//
// Precision. The reference multiplies f32 activations with widened f16 weights and accumulates in f32, and
// greedy decoding on a random-init model has to reproduce its token choices, so activations are NOT
// rounded to f16: x is split as x = hi + lo with hi = f16(x), lo = f16(x - hi), and every k-step issues two MMAs
// into the same f32 accumulator, hi*W and lo*W. The pair carries 22 significant bits while lo is a normal f16,
// i.e. for |x| above about 2^-4; below that lo falls into the f16 subnormals (spacing 2^-24), so what the split
// guarantees for every x is an ABSOLUTE error of at most 2^-25 per element (relative 3e-5 for an activation
// near 1e-3). The weights are used as stored, the products are exact, the accumulation is f32: the result
// differs from the reference only by summation order and that truncation of x.
//
// bf16 models (ingot_linear_ws_create_bf16). The same kernel on bf16 weights with the activations as one bf16 plane (plain
// bf16 products) or as a hi + lo pair (16 significant bits, for products that feed a recurrence's gates); the number of
// planes is chosen per product. Rows of any length that is a multiple of 8 are accepted (the last k-step is zero-filled
// by TMA), and a matrix may be block-diagonal: output tiles of block b then read the k_block activation columns that
// start at b * k_block.
//
// Grouped products (ingot_grouped_tc_run). One matrix per group of rows - the experts of a mixture - in one launch: the rows are
// sorted by group, group g's rows are a run of the activation matrix that starts anywhere, and its matrix is the g-th of a stack. A
// CTA finds its group and row tile from the run starts on the device; boxes that reach into the next run are multiplied along and
// not stored. The activation of an expert is folded into the epilogue, which then writes the bf16 operand of the next product.
//
// Kernel. One CTA = 128 tokens x 128 outputs over a slice of k (split-k fills the GPU when there are few
// output tiles; slices go to a scratch and are summed in slice order, by a small kernel or by the kernel
// that consumes the product, so results are reproducible). 6 warps: warp 0 streams [128 rows][64 k] boxes of hi, lo and W (128-byte swizzle, 48 KB per
// stage, 4 stages) with TMA; warp 1 issues tcgen05.mma (kind::f16, M = N = 128, K = 16; all lanes walk the
// loop, one elected lane issues); warps 2-5 read the 128x128 f32 accumulator out of tensor memory, one
// thread per token row. Rows past n_tok and outputs past n_out are zero-filled by TMA and not stored.
// Every mbarrier wait is bounded; on expiry the CTA raises the workspace's status word and leaves.
#include "grouped_linear.h"
#include "../csrc/sm100_ptx.cuh"

#include <cuda_bf16.h>
#include <cuda_fp16.h>

#include <algorithm>
#include <map>
#include <mutex>
#include <tuple>

namespace {

using namespace ingot_sm100;

constexpr int kBM = 128, kBK = 64;  // outputs per CTA (kBN): 128, or 256 (a quarter less L2 traffic per output with one plane)
constexpr int kGroupM = 16;         // token tiles that sweep the weight matrix together (see the tile order in the kernel)
constexpr int kMaxStages = 6;
constexpr int kBoxBytes = 128 * kBK * 2;        // 16 KB: 128 rows x 64 f16
constexpr int kThreads = 192;
template <int kPlanes, int kBN>
struct Ring {
    static constexpr int kWBytes = kBN * kBK * 2;                      // the W box: kBN rows
    static constexpr int kStageBytes = kPlanes * kBoxBytes + kWBytes;  // hi(, lo), W
    static constexpr int kStages = 196608 / kStageBytes;               // 192 KB ring: 4 stages of 48 KB or 6 of 32 KB
    static constexpr int kOffBar = kStages * kStageBytes;
    static constexpr int kSmemBytes = kOffBar + 256 + 1024;            // barriers + alignment slack
    static_assert(kStages <= kMaxStages, "barrier arrays");
};
constexpr uint32_t idesc_f16(int kBN) { return (1u << 4) | ((uint32_t)(kBN >> 3) << 17) | ((uint32_t)(kBM >> 4) << 24); }  // f16 x f16 -> f32, both K-major
constexpr uint32_t kIdescBF16 = (1u << 7) | (1u << 10);  // bf16 x bf16 -> f32
constexpr unsigned long long kWaitLimitNs = 2000000000ull;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

// Programmatic dependent launch, as in the attention kernels: every kernel of the batched path lets its successor
// start early (launch_dependents at its top) and waits for its predecessor before it touches anything the predecessor
// wrote; launch latency and per-CTA set-up then overlap the predecessor's tail. INGOT_NO_PDL=1: plain stream order.
#define LINEAR_PDL_TRIGGER() asm volatile("griddepcontrol.launch_dependents;" ::: "memory")
#define LINEAR_PDL_WAIT() asm volatile("griddepcontrol.wait;" ::: "memory")
template <typename... KArgs, typename... Args>
static cudaError_t launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args&&... args) {
    static const bool use_pdl = getenv("INGOT_NO_PDL") == nullptr;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = use_pdl ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);
}

struct Bars {
    uint64_t full[kMaxStages];
    uint64_t empty[kMaxStages];
    uint64_t done;
    uint32_t tmem_base;
    uint32_t abort_flag;
};

// One launch covers up to three weight matrices that read the same activations (q/k/v, gate/up): grid.x runs over
// the token tiles and the output tiles of all of them, tile_end[m] being the running total of tiles up to and including matrix m.
struct GemmParams {
    float* out;           // [n_tok][n_out] (single matrix only)
    float* partial[3];    // per matrix: [n_split][n_tok][n_out] when n_split > 1 or to_partial
    int* status;
    int n_tok, k_steps, n_split, accumulate;
    int n_out[3], tile_end[3];
    int tiles_n, tiles_m;
    int a_bytes;  // of one activation box: 128 rows, or fewer for a single short token tile
    uint32_t idesc;
    int rows_per_block, k_block, tiles_per_block;  // block-diagonal matrix (rows_per_block > 0, count == 1)
    // grouped: run starts [n_groups + 1] of the rows; out rows are the sorted rows
    const int32_t* group_start;
    int n_groups;
    const float* row_scale;                // epilogue: accumulator * row_scale[row] (null: none), then act
    int act;                               // 1: square of relu, 2: silu(gate) * up (INGOT_ACT_*)
    __nv_bfloat16 *out_hi, *out_lo;        // bf16 plane(s) [rows][n_out] instead of f32
    __half* out_half;                      // f16 instead of f32: row stride half_ld, block b's columns from b * half_block on
    int half_ld, half_block;
    int to_partial;  // write the slice(s) to `partial` even when there is only one (a consumer kernel sums them)
};

template <int kPlanes, int kBN, bool kGrouped>
__global__ void __launch_bounds__(kThreads, 1)
linear_sm100_kernel(const __grid_constant__ CUtensorMap map_hi, const __grid_constant__ CUtensorMap map_lo,
                    const __grid_constant__ CUtensorMap map_w0, const __grid_constant__ CUtensorMap map_w1,
                    const __grid_constant__ CUtensorMap map_w2, const GemmParams p) {
    using R = Ring<kPlanes, kBN>;
    constexpr int kStages = R::kStages, kStageBytes = R::kStageBytes, kOffBar = R::kOffBar;
    constexpr uint32_t kTmemCols = kBN;
    constexpr int kOffW = kPlanes * kBoxBytes;
    extern __shared__ unsigned char smem_dyn[];
    LINEAR_PDL_TRIGGER();
    const uint32_t smem_base = (smem_u32(smem_dyn) + 1023u) & ~1023u;
    unsigned char* smem_al = smem_dyn + (smem_base - smem_u32(smem_dyn));
    Bars* bars = reinterpret_cast<Bars*>(smem_al + kOffBar);
    volatile uint32_t* abort_flag = &bars->abort_flag;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int warp_u = __shfl_sync(0xffffffffu, warp, 0);
    // Tile order: kGroupM token tiles walk the output tiles together, so that CTAs that run at the same time share weight
    // boxes and the weight matrix comes out of HBM once per kGroupM * 128 tokens instead of once per 128.
    const int group_tiles = kGroupM * p.tiles_n, grp = (int)blockIdx.x / group_tiles, in_grp = (int)blockIdx.x - grp * group_tiles;
    const int group_m = min(kGroupM, p.tiles_m - grp * kGroupM);
    const int tile_n = in_grp / group_m, tile_m = grp * kGroupM + in_grp - tile_n * group_m;
    const int mat = (tile_n >= p.tile_end[0]) + (tile_n >= p.tile_end[1]);  // warp-uniform
    const CUtensorMap* const map_w_p = mat == 0 ? &map_w0 : mat == 1 ? &map_w1 : &map_w2;
    const int mat_n_out = mat == 0 ? p.n_out[0] : mat == 1 ? p.n_out[1] : p.n_out[2];
    // grouped: which group's which row tile this is, 32 groups at a time
    int group = 0, group_m0 = 0, group_end = 0;
    if (kGrouped) {
        LINEAR_PDL_WAIT();  // the runs come from a kernel before
        int tile = tile_m;
        bool found = false;
        for (int g0 = 0; g0 < p.n_groups && !found; g0 += 32) {
            const int mine = g0 + lane;
            const int a = mine < p.n_groups ? p.group_start[mine] : 0, b = mine < p.n_groups ? p.group_start[mine + 1] : 0;
            const int n = (b - a + kBM - 1) / kBM;
            int upto = n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, upto, o);
                if (lane >= o) upto += v;
            }
            const unsigned hit = __ballot_sync(0xffffffffu, tile < upto);
            if (hit) {
                const int src = __ffs(hit) - 1;
                const int local = tile - (__shfl_sync(0xffffffffu, upto, src) - __shfl_sync(0xffffffffu, n, src));
                group = g0 + src;
                group_m0 = __shfl_sync(0xffffffffu, a, src) + local * kBM;
                group_end = __shfl_sync(0xffffffffu, b, src);
                found = true;
            } else {
                tile -= __shfl_sync(0xffffffffu, upto, 31);
            }
        }
        if (!found) return;  // the grid covers the most row tiles there can be
    }
    const int row_end = kGrouped ? group_end : p.n_tok;
    const int blk = p.tiles_per_block > 0 ? tile_n / p.tiles_per_block : 0;
    const int col_end = p.tiles_per_block > 0 ? (blk + 1) * p.rows_per_block : mat_n_out;
    const int a_k0 = blk * p.k_block;  // first activation column of this tile's products
    float* const mat_partial = mat == 0 ? p.partial[0] : mat == 1 ? p.partial[1] : p.partial[2];
    const int n0 = p.tiles_per_block > 0 ? blk * p.rows_per_block + (tile_n - blk * p.tiles_per_block) * kBN
                                         : (tile_n - (mat == 0 ? 0 : mat == 1 ? p.tile_end[0] : p.tile_end[1])) * kBN;
    const int m0 = kGrouped ? group_m0 : tile_m * kBM, split = blockIdx.z;
    const int w_row0 = kGrouped ? group * mat_n_out + n0 : n0;  // row of the weight matrix, or of the stack of matrices
    const int ks_begin = (int)((long long)p.k_steps * split / p.n_split);
    const int ks_end = (int)((long long)p.k_steps * (split + 1) / p.n_split);
    const int n_it = ks_end - ks_begin;

    if (threadIdx.x == 0) {
        for (int s = 0; s < kStages; s++) { mbar_init(smem_u32(&bars->full[s]), 1); mbar_init(smem_u32(&bars->empty[s]), 1); }
        mbar_init(smem_u32(&bars->done), 1);
        bars->abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&bars->tmem_base)), "r"(kTmemCols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = bars->tmem_base;
    // Barriers and tensor memory are this CTA's own and the weights never depend on the kernel before: the W boxes of
    // the first ring stages are requested now, the activation boxes (and, under accumulate, the output) only after the
    // wait for the predecessor. A stage's barrier is armed once for all three boxes.
    const uint32_t stage_tx = kPlanes * p.a_bytes + R::kWBytes;
    const int n_pre = min(n_it, kStages);
    if (warp_u == 0 && lane == 0) {
        for (int it = 0; it < n_pre; it++) {
            const uint32_t full = smem_u32(&bars->full[it]);
            mbar_expect_tx(full, stage_tx);
            tma_load_2d(smem_base + it * kStageBytes + kOffW, map_w_p, (ks_begin + it) * kBK, w_row0, full);
        }
    }
    if (!kGrouped) LINEAR_PDL_WAIT();

    if (warp_u == 0) {
        // ---------------- TMA producer ----------------
        int armed = 0;
        bool ok = true;
        for (int it = 0; it < n_it && ok; it++) {
            const int s = it % kStages;
            const uint32_t full = smem_u32(&bars->full[s]);
            if (lane == 0) {
                const uint32_t dst = smem_base + s * kStageBytes;
                const int k = (ks_begin + it) * kBK;
                if (it < n_pre) {  // first use of the slot: armed and its W box requested before the wait above
                    tma_load_2d(dst, &map_hi, a_k0 + k, m0, full);
                    if (kPlanes > 1) tma_load_2d(dst + kBoxBytes, &map_lo, a_k0 + k, m0, full);
                } else {
                    ok = mbar_wait(smem_u32(&bars->empty[s]), (uint32_t)(((it / kStages) & 1) ^ 1), abort_flag, kWaitLimitNs);
                    if (ok) {
                        mbar_expect_tx(full, stage_tx);
                        tma_load_2d(dst, &map_hi, a_k0 + k, m0, full);
                        if (kPlanes > 1) tma_load_2d(dst + kBoxBytes, &map_lo, a_k0 + k, m0, full);
                        tma_load_2d(dst + kOffW, map_w_p, k, w_row0, full);
                    }
                }
            }
            ok = __shfl_sync(0xffffffffu, ok, 0);
            if (ok) armed = it + 1;
        }
        if (!ok && lane == 0) {
            // copies already issued must land before the CTA's shared memory is released
            for (int it = max(0, armed - kStages); it < armed; it++) {
                const uint64_t t0 = globaltimer_ns();
                while (!mbar_try_wait(smem_u32(&bars->full[it % kStages]), (uint32_t)((it / kStages) & 1)) &&
                       globaltimer_ns() - t0 < 100000000ull) {}
            }
        }
    } else if (warp_u == 1) {
        // ---------------- MMA issuer ----------------
        bool ok = true;
        for (int it = 0; it < n_it && ok; it++) {
            const int s = it % kStages;
            ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(&bars->full[s]), (uint32_t)((it / kStages) & 1), abort_flag, kWaitLimitNs)) != 0;
            if (!ok) break;
            tc_fence_after();
            if (elect_one()) {
                const uint32_t a_hi = smem_base + s * kStageBytes, a_lo = a_hi + kBoxBytes, b = a_hi + kOffW;
#pragma unroll
                for (int ks = 0; ks < kBK / 16; ks++)
                    tc_mma_ss(tmem, make_desc(a_hi + ks * 32, 16, 1024), make_desc(b + ks * 32, 16, 1024), p.idesc, (it > 0 || ks > 0) ? 1u : 0u);
                if (kPlanes > 1) {
#pragma unroll
                    for (int ks = 0; ks < kBK / 16; ks++)
                        tc_mma_ss(tmem, make_desc(a_lo + ks * 32, 16, 1024), make_desc(b + ks * 32, 16, 1024), p.idesc, 1u);
                }
                tc_commit(smem_u32(&bars->empty[s]));
                if (it == n_it - 1) tc_commit(smem_u32(&bars->done));
            }
            __syncwarp();
        }
    } else {
        // ---------------- epilogue: accumulator -> global, one thread per token row ----------------
        const int lg = warp & 3;  // the tensor-memory lane group this warp may read
        const int row = m0 + lg * 32 + lane;
        bool ok = n_it > 0 && mbar_wait(smem_u32(&bars->done), 0, abort_flag, kWaitLimitNs);
        ok = __all_sync(0xffffffffu, ok) != 0;
        const bool split_k = p.n_split > 1 || p.to_partial;
        if (ok) {
            tc_fence_after();
            float* dst = (split_k ? mat_partial + (size_t)split * p.n_tok * mat_n_out : p.out) + (size_t)row * mat_n_out + n0;
            const bool add = !split_k && p.accumulate;
            const float scale = p.row_scale && row < row_end ? p.row_scale[row] : 1.0f;
            if (kGrouped && p.act == 2) {
                // Runs of 32 gate columns, each followed by the 32 up columns of the same outputs: scale * silu(gate) * up, half as wide.
                const int half_out = mat_n_out / 2;
#pragma unroll
                for (int c = 0; c < kBN / 64; c++) {
                    float g[32], u[32];
                    tmem_ld32(tmem + ((uint32_t)(lg * 32) << 16) + c * 64, g);
                    tmem_ld32(tmem + ((uint32_t)(lg * 32) << 16) + c * 64 + 32, u);
                    tmem_wait_ld();
                    if (row >= row_end || n0 + c * 64 >= mat_n_out) continue;
                    const size_t at = (size_t)row * half_out + n0 / 2 + c * 32;
#pragma unroll
                    for (int i = 0; i < 32; i += 8) {
                        __nv_bfloat162 h[4], l[4];
#pragma unroll
                        for (int e = 0; e < 4; e++) {
                            const float a = g[i + 2 * e], b = g[i + 2 * e + 1];
                            const float x = a / (1.0f + expf(-a)) * u[i + 2 * e] * scale, y = b / (1.0f + expf(-b)) * u[i + 2 * e + 1] * scale;
                            h[e] = __floats2bfloat162_rn(x, y);
                            l[e] = __floats2bfloat162_rn(x - __low2float(h[e]), y - __high2float(h[e]));
                        }
                        *reinterpret_cast<uint4*>(p.out_hi + at + i) = *reinterpret_cast<const uint4*>(h);
                        if (p.out_lo) *reinterpret_cast<uint4*>(p.out_lo + at + i) = *reinterpret_cast<const uint4*>(l);
                    }
                }
            } else {
#pragma unroll
                for (int c = 0; c < kBN / 32; c++) {
                    float v[32];
                    tmem_ld32(tmem + ((uint32_t)(lg * 32) << 16) + c * 32, v);
                    tmem_wait_ld();
                    if (row < row_end) {
                        if (kGrouped && (p.row_scale || p.act)) {
#pragma unroll
                            for (int i = 0; i < 32; i++) {
                                v[i] *= scale;
                                if (p.act == 1) v[i] = v[i] > 0.f ? v[i] * v[i] : 0.f;
                            }
                        }
                        if (kGrouped && p.out_hi) {  // n_out is a multiple of 8
#pragma unroll
                            for (int i = 0; i < 32; i += 8) {
                                const int col = n0 + c * 32 + i;
                                if (col >= col_end) break;
                                const size_t at = (size_t)row * mat_n_out + col;
                                __nv_bfloat162 h[4], l[4];
#pragma unroll
                                for (int e = 0; e < 4; e++) {
                                    h[e] = __floats2bfloat162_rn(v[i + 2 * e], v[i + 2 * e + 1]);
                                    l[e] = __floats2bfloat162_rn(v[i + 2 * e] - __low2float(h[e]), v[i + 2 * e + 1] - __high2float(h[e]));
                                }
                                *reinterpret_cast<uint4*>(p.out_hi + at) = *reinterpret_cast<const uint4*>(h);
                                if (p.out_lo) *reinterpret_cast<uint4*>(p.out_lo + at) = *reinterpret_cast<const uint4*>(l);
                            }
                        } else if (!kGrouped && p.out_half) {  // n_out and the blocks are multiples of 8
#pragma unroll
                            for (int i = 0; i < 32; i += 8) {
                                const int col = n0 + c * 32 + i;
                                if (col >= col_end) break;
                                __half2 h[4];
#pragma unroll
                                for (int e = 0; e < 4; e++)
                                    h[e] = __floats2half2_rn(fminf(fmaxf(v[i + 2 * e], -65504.f), 65504.f), fminf(fmaxf(v[i + 2 * e + 1], -65504.f), 65504.f));
                                *reinterpret_cast<uint4*>(p.out_half + (size_t)row * p.half_ld + blk * p.half_block + (col - blk * p.rows_per_block)) = *reinterpret_cast<const uint4*>(h);
                            }
                        } else {
#pragma unroll
                            for (int i = 0; i < 32; i += 4) {
                                const int col = n0 + c * 32 + i;
                                if (col + 3 < col_end) {
                                    float4* d4 = reinterpret_cast<float4*>(dst + c * 32 + i);
                                    float4 o = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
                                    if (add) { const float4 old = *d4; o.x += old.x; o.y += old.y; o.z += old.z; o.w += old.w; }
                                    *d4 = o;
                                } else {
                                    for (int e = 0; e < 4; e++)
                                        if (col + e < col_end) dst[c * 32 + i + e] = add ? dst[c * 32 + i + e] + v[i + e] : v[i + e];
                                }
                            }
                        }
                    }
                }
            }
        }
    }

    tc_fence_before();
    __syncthreads();
    if (threadIdx.x == 0 && *abort_flag) atomicOr(p.status, 1);
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kTmemCols) : "memory");
    }
}

// out (+)= sum over the k slices, in slice order
__global__ void splitk_reduce_kernel(float* out, const float* partial, int n_split, size_t n, int accumulate) {
    LINEAR_PDL_TRIGGER();
    LINEAR_PDL_WAIT();
    const size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i >= n) return;
    float4 acc = accumulate ? *reinterpret_cast<const float4*>(out + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < n_split; s++) {
        const float4 v = *reinterpret_cast<const float4*>(partial + (size_t)s * n + i);
        acc.x += v.x; acc.y += v.y; acc.z += v.z; acc.w += v.w;
    }
    *reinterpret_cast<float4*>(out + i) = acc;
}

// How f32 activations become MMA operands: an f16 pair hi = f16(x), lo = f16(x - hi), one bf16 plane, or a bf16 pair.
enum : int { kActF16Pair = 0, kActBF16 = 1, kActBF16Pair = 2 };
template <int kAct>
__device__ __forceinline__ void store_split4(__half* hi, __half* lo, size_t i, const float (&f)[4]) {
    if (kAct == kActF16Pair) {
        __half h[4], l[4];
#pragma unroll
        for (int e = 0; e < 4; e++) {
            h[e] = __float2half_rn(f[e]);
            l[e] = __float2half_rn(f[e] - __half2float(h[e]));
        }
        *reinterpret_cast<uint2*>(hi + i) = *reinterpret_cast<const uint2*>(h);
        *reinterpret_cast<uint2*>(lo + i) = *reinterpret_cast<const uint2*>(l);
    } else {
        __nv_bfloat16 h[4], l[4];
#pragma unroll
        for (int e = 0; e < 4; e++) {
            h[e] = __float2bfloat16_rn(f[e]);
            l[e] = __float2bfloat16_rn(f[e] - __bfloat162float(h[e]));
        }
        *reinterpret_cast<uint2*>(hi + i) = *reinterpret_cast<const uint2*>(h);
        if (kAct == kActBF16Pair) *reinterpret_cast<uint2*>(lo + i) = *reinterpret_cast<const uint2*>(l);
    }
}

// x rows are x_ld floats apart, the planes' rows n; grid.y = row
template <int kAct>
__global__ void split_act_kernel(__half* hi, __half* lo, const float* x, int x_ld, int n) {
    LINEAR_PDL_TRIGGER();
    LINEAR_PDL_WAIT();
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i >= n) return;
    const float4 v = *reinterpret_cast<const float4*>(x + (size_t)blockIdx.y * x_ld + i);
    const float f[4] = {v.x, v.y, v.z, v.w};
    store_split4<kAct>(hi, lo, (size_t)blockIdx.y * n + i, f);
}

// hi/lo of rmsnorm(x) = x * rsqrt(mean(x^2) + eps) * w, one CTA per token row (ops::rmsnorm, src/ops.cpp:227-232,
// with the same expression order as the standalone norm kernel, so the split sees the same f32 values).
// The mean is taken over n_mean of the row's n floats (rows zero-padded to an aligned length).
template <int kAct>
__global__ void rmsnorm_split_kernel(__half* hi, __half* lo, const float* x, const float* w, int n, int n_mean, float eps) {
    LINEAR_PDL_TRIGGER();
    LINEAR_PDL_WAIT();
    __shared__ float red[32];
    const float* xr = x + (size_t)blockIdx.x * n;
    constexpr int kKeep = 4;  // float4s of the row a thread keeps between the two passes
    float4 kept[kKeep];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < kKeep; k++) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        kept[k] = i < n ? *reinterpret_cast<const float4*>(xr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int k = 0; k < kKeep; k++) { ss += kept[k].x * kept[k].x; ss += kept[k].y * kept[k].y; ss += kept[k].z * kept[k].z; ss += kept[k].w * kept[k].w; }
    for (int i = (threadIdx.x + kKeep * blockDim.x) * 4; i < n; i += blockDim.x * 4) {
        const float4 v = *reinterpret_cast<const float4*>(xr + i);
        ss += v.x * v.x; ss += v.y * v.y; ss += v.z * v.z; ss += v.w * v.w;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    if (threadIdx.x < 32) {
        float v = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0.f;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
        if (threadIdx.x == 0) red[0] = 1.0f / sqrtf(v / float(n_mean) + eps);
    }
    __syncthreads();
    const float scale = red[0];
    auto put = [&](int i, const float4& v) {
        const float4 g = *reinterpret_cast<const float4*>(w + i);
        const float f[4] = {v.x * scale * g.x, v.y * scale * g.y, v.z * scale * g.z, v.w * scale * g.w};
        store_split4<kAct>(hi, lo, (size_t)blockIdx.x * n + i, f);
    };
#pragma unroll
    for (int k = 0; k < kKeep; k++) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (i < n) put(i, kept[k]);
    }
    for (int i = (threadIdx.x + kKeep * blockDim.x) * 4; i < n; i += blockDim.x * 4) put(i, *reinterpret_cast<const float4*>(xr + i));
}

// Consumers of k-slice partials [n_split][n_tok][n_out]: the sum over slices (always in slice order) is folded into
// the kernel that needs the result, so a split-k GEMM costs no reduction launch of its own.
struct Slices {
    const float* base;
    int n_split;
};
__device__ __forceinline__ float4 sum_slices(const Slices& p, size_t idx, size_t slice_elems, float4 acc) {
    for (int sl = 0; sl < p.n_split; sl++) {
        const float4 v = *reinterpret_cast<const float4*>(p.base + sl * slice_elems + idx);
        acc.x += v.x; acc.y += v.y; acc.z += v.z; acc.w += v.w;
    }
    return acc;
}

// Up to three plain outputs (q, k, v): out_m = sum of its slices. grid.y selects the output.
struct FinishGroup {
    Slices in[3];
    float* out[3];
    int n_out[3];
};
__global__ void finish_group_kernel(const FinishGroup g, int n_tok) {
    LINEAR_PDL_TRIGGER();
    LINEAR_PDL_WAIT();
    const int m = blockIdx.y;
    const Slices in = m == 0 ? g.in[0] : m == 1 ? g.in[1] : g.in[2];
    float* out = m == 0 ? g.out[0] : m == 1 ? g.out[1] : g.out[2];
    const size_t n = (size_t)n_tok * (m == 0 ? g.n_out[0] : m == 1 ? g.n_out[1] : g.n_out[2]);
    const size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i >= n) return;
    *reinterpret_cast<float4*>(out + i) = sum_slices(in, i, n, make_float4(0.f, 0.f, 0.f, 0.f));
}

// x[t][:] += sum of slices (the residual add of wo / down), then, if norm_w is given, hi/lo of rmsnorm(x[t]) for the
// next projections. One CTA per token.
// pair_rows (may be null): rows of another branch that go into the sum, token t's at row_of[t * top + k] (row_of null: t).
template <int kAct>
__global__ void finish_residual_norm_kernel(float* x, const Slices in, __half* hi, __half* lo, const float* norm_w, int n, int n_mean, int n_tok,
                                            float eps, const float* pair_rows, const int32_t* row_of, int top) {
    __shared__ float red[32];
    LINEAR_PDL_TRIGGER();
    LINEAR_PDL_WAIT();
    const size_t row = (size_t)blockIdx.x * n;
    const size_t slice = (size_t)n_tok * n;
    float ss = 0.f;
    for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
        float4 v = sum_slices(in, row + i, slice, *reinterpret_cast<const float4*>(x + row + i));
        for (int k = 0; k < top; k++) {
            const float4 a = *reinterpret_cast<const float4*>(pair_rows + (row_of ? (size_t)row_of[blockIdx.x * top + k] : (size_t)blockIdx.x) * n + i);
            v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w;
        }
        *reinterpret_cast<float4*>(x + row + i) = v;
        ss += v.x * v.x; ss += v.y * v.y; ss += v.z * v.z; ss += v.w * v.w;
    }
    if (norm_w == nullptr) return;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    if (threadIdx.x < 32) {
        float v = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0.f;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
        if (threadIdx.x == 0) red[0] = 1.0f / sqrtf(v / float(n_mean) + eps);
    }
    __syncthreads();
    const float scale = red[0];
    for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
        const float4 v = *reinterpret_cast<const float4*>(x + row + i), g = *reinterpret_cast<const float4*>(norm_w + i);
        const float f[4] = {v.x * scale * g.x, v.y * scale * g.y, v.z * scale * g.z, v.w * scale * g.w};
        store_split4<kAct>(hi, lo, row + i, f);
    }
}

// hi/lo of silu(sum of gate slices) * (sum of up slices)
__global__ void finish_swiglu_kernel(__half* hi, __half* lo, const Slices gate, const Slices up, size_t n) {
    LINEAR_PDL_TRIGGER();
    LINEAR_PDL_WAIT();
    const size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i >= n) return;
    const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 g = sum_slices(gate, i, n, z), u = sum_slices(up, i, n, z);
    const float f[4] = {g.x / (1.0f + expf(-g.x)) * u.x, g.y / (1.0f + expf(-g.y)) * u.y, g.z / (1.0f + expf(-g.z)) * u.z,
                        g.w / (1.0f + expf(-g.w)) * u.w};
    store_split4<kActF16Pair>(hi, lo, i, f);
}

// One or two bf16 planes of act(gate) * up, where one product of width 2 n holds both: gate = columns 0..n-1, up = columns n..2n-1.
// act: 0 silu, 1 the tanh form of gelu. grid.y = row.
template <int kAct>
__global__ void finish_gated_kernel(__half* hi, __half* lo, const Slices in, int n, size_t slice, int act) {
    LINEAR_PDL_TRIGGER();
    LINEAR_PDL_WAIT();
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i >= n) return;
    const size_t row = (size_t)blockIdx.y * 2 * n;
    const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 g = sum_slices(in, row + i, slice, z), u = sum_slices(in, row + n + i, slice, z);
    const float gv[4] = {g.x, g.y, g.z, g.w}, uv[4] = {u.x, u.y, u.z, u.w};
    float f[4];
#pragma unroll
    for (int e = 0; e < 4; e++) {
        const float t = gv[e];
        f[e] = (act == 0 ? t / (1.0f + expf(-t)) : 0.5f * t * (1.0f + tanhf(0.7978845608028654f * (t + 0.044715f * t * t * t)))) * uv[e];
    }
    store_split4<kAct>(hi, lo, (size_t)blockIdx.y * n + i, f);
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

// f16 or bf16 matrix [rows][cols] row-major, boxes of box_rows rows x 64 columns, 128-byte swizzle, zero fill outside
bool make_map(CUtensorMap* map, const void* base, int rows, int cols, int box_rows = 128, bool bf16 = false) {
    EncodeTiledFn fn = encode_fn();
    if (!fn) return false;
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)cols * 2};
    const cuuint32_t box[2] = {(cuuint32_t)kBK, (cuuint32_t)box_rows};
    const cuuint32_t elem[2] = {1, 1};
    return fn(map, bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 2, const_cast<void*>(base), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

}  // namespace

struct ingot_linear_ws {
    __half* hi = nullptr;
    __half* lo = nullptr;
    float* partial = nullptr;
    int* status = nullptr;
    size_t act_elems = 0, partial_floats = 0;  // partial_floats: per slot; kSlots slots
    int slot_split[3] = {0, 0, 0};             // slices the last GEMM into each slot produced
    int slot_out[3] = {0, 0, 0};               // and its output width
    int num_sms = 0;
    bool bf16 = false;
    int n_slots = 3;
    int planes = 2;                            // of the prepared activations
    int box_rows = 128;
    int prepared_tok = 0, prepared_in = 0;
    CUtensorMap map_hi, map_lo;
    std::map<std::tuple<const void*, int, int, int>, CUtensorMap> w_maps;  // one per weight matrix (and per row count of grouped activations)
};

// (Re)builds the activation tensor maps when the prepared shape changes.
static cudaError_t set_prepared(ingot_linear_ws* ws, int n_in, int n_tok) {
    if (ws->prepared_tok != n_tok || ws->prepared_in != n_in) {
        // A batch of few tokens fetches only its own rows (whole 8-row swizzle groups) of the 128 a tile has. What the other rows of
        // the tile hold is multiplied along and never stored: rows of a product do not mix.
        ws->box_rows = n_tok >= 128 ? 128 : (n_tok + 7) / 8 * 8;
        if (!make_map(&ws->map_hi, ws->hi, n_tok, n_in, ws->box_rows, ws->bf16) || !make_map(&ws->map_lo, ws->lo, n_tok, n_in, ws->box_rows, ws->bf16))
            return cudaErrorUnknown;
        ws->prepared_tok = n_tok;
        ws->prepared_in = n_in;
    }
    return cudaGetLastError();
}

extern "C" {

static cudaError_t ws_create(ingot_linear_ws** out, size_t act_elems, size_t partial_floats, int n_slots, bool bf16) {
    *out = nullptr;
    ingot_linear_ws* ws = new ingot_linear_ws();
    ws->act_elems = act_elems;
    ws->partial_floats = partial_floats;
    ws->n_slots = n_slots;
    ws->bf16 = bf16;
    ws->planes = bf16 ? 1 : 2;
    int dev = 0;
    cudaError_t e;
    if ((e = cudaGetDevice(&dev)) != cudaSuccess ||
        (e = cudaDeviceGetAttribute(&ws->num_sms, cudaDevAttrMultiProcessorCount, dev)) != cudaSuccess ||
        (e = cudaMalloc(&ws->hi, ws->act_elems * 2)) != cudaSuccess || (e = cudaMalloc(&ws->lo, ws->act_elems * 2)) != cudaSuccess ||
        // zero-filled: padding columns that no producer writes must be finite, they meet zero weights
        (e = cudaMemset(ws->hi, 0, ws->act_elems * 2)) != cudaSuccess || (e = cudaMemset(ws->lo, 0, ws->act_elems * 2)) != cudaSuccess ||
        (e = cudaMalloc(&ws->partial, n_slots * ws->partial_floats * 4)) != cudaSuccess || (e = cudaMalloc(&ws->status, sizeof(int))) != cudaSuccess ||
        (e = cudaMemset(ws->status, 0, sizeof(int))) != cudaSuccess ||
        (e = cudaFuncSetAttribute(linear_sm100_kernel<2, 128, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, Ring<2, 128>::kSmemBytes)) != cudaSuccess ||
        (e = cudaFuncSetAttribute(linear_sm100_kernel<1, 128, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, Ring<1, 128>::kSmemBytes)) != cudaSuccess ||
        (e = cudaFuncSetAttribute(linear_sm100_kernel<1, 256, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, Ring<1, 256>::kSmemBytes)) != cudaSuccess ||
        (e = cudaFuncSetAttribute(linear_sm100_kernel<2, 128, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, Ring<2, 128>::kSmemBytes)) != cudaSuccess ||
        (e = cudaFuncSetAttribute(linear_sm100_kernel<1, 128, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, Ring<1, 128>::kSmemBytes)) != cudaSuccess ||
        (e = cudaFuncSetAttribute(linear_sm100_kernel<1, 256, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, Ring<1, 256>::kSmemBytes)) != cudaSuccess) {
        cudaFree(ws->hi); cudaFree(ws->lo); cudaFree(ws->partial); cudaFree(ws->status);
        delete ws;
        return e;
    }
    *out = ws;
    return cudaSuccess;
}

// max_tok x max_in: the largest activation matrix that will be prepared; also the largest output (tokens x width).
cudaError_t ingot_linear_ws_create(ingot_linear_ws** out, int max_tok, int max_in) {
    // k-slice partials: three slots, each at least two full-width slices of the largest batch (the hi-plane and the
    // lo-plane product of a quantised matrix), 24 MB or more
    const size_t act = (size_t)max_tok * max_in;
    return ws_create(out, act, std::max((size_t)6 << 20, 2 * act), 3, false);
}

// bf16 weights: one partial slot that holds at least one slice of max_tok x max_out.
cudaError_t ingot_linear_ws_create_bf16(ingot_linear_ws** out, int max_tok, int max_in, int max_out) {
    return ws_create(out, (size_t)max_tok * max_in, std::max((size_t)6 << 20, (size_t)max_tok * max_out), 1, true);
}

void ingot_linear_ws_destroy(ingot_linear_ws* ws) {
    if (!ws) return;
    cudaFree(ws->hi); cudaFree(ws->lo); cudaFree(ws->partial); cudaFree(ws->status);
    delete ws;
}

// Whether a projection of this shape can take the tensor-core path.
int ingot_linear_tc_supported(const ingot_linear_ws* ws, int w_is_f16, int n_in, int n_out, int n_tok) {
    if (!ws || !encode_fn() || n_tok < (ws->bf16 ? 2 : 16) || n_out % 4 != 0 || (size_t)n_tok * n_in > ws->act_elems) return 0;
    return ws->bf16 ? n_in % 8 == 0 : w_is_f16 && n_in % kBK == 0;
}

// Row length the planes may have: whole k-steps of f16, any multiple of 8 of bf16.
static bool act_shape_ok(const ingot_linear_ws* ws, int n_in, int n_tok) {
    return (size_t)n_tok * n_in <= ws->act_elems && n_in % (ws->bf16 ? 8 : kBK) == 0;
}

// Splits x [n_tok][n_in] f32 into the workspace's hi/lo f16 matrices; the following ingot_linear_tc_run calls use them.
cudaError_t ingot_linear_tc_prepare(ingot_linear_ws* ws, const float* x, int n_in, int n_tok, cudaStream_t s) {
    if (!act_shape_ok(ws, n_in, n_tok) || ws->bf16) return cudaErrorInvalidValue;
    cudaError_t le = launch_pdl(split_act_kernel<kActF16Pair>, dim3((unsigned)((n_in / 4 + 255) / 256), n_tok), dim3(256), 0, s, ws->hi, ws->lo, x, n_in, n_in);
    if (le != cudaSuccess) return le;
    return set_prepared(ws, n_in, n_tok);
}

// bf16 workspace: rows of x are x_ld floats apart; planes 1 or 2.
cudaError_t ingot_linear_tc_prepare_bf16(ingot_linear_ws* ws, const float* x, int x_ld, int n_in, int n_tok, int planes, cudaStream_t s) {
    if (!act_shape_ok(ws, n_in, n_tok) || !ws->bf16 || x_ld % 4 != 0) return cudaErrorInvalidValue;
    const dim3 grid((unsigned)((n_in / 4 + 255) / 256), n_tok);
    cudaError_t le = planes > 1 ? launch_pdl(split_act_kernel<kActBF16Pair>, grid, dim3(256), 0, s, ws->hi, ws->lo, x, x_ld, n_in)
                                : launch_pdl(split_act_kernel<kActBF16>, grid, dim3(256), 0, s, ws->hi, ws->lo, x, x_ld, n_in);
    if (le != cudaSuccess) return le;
    ws->planes = planes > 1 ? 2 : 1;
    return set_prepared(ws, n_in, n_tok);
}

// The planes themselves ([n_tok][n_in] bf16, row-contiguous) for kernels that write their output as the next product's
// operand, and the declaration that they have been (or, in stream order, will have been) written.
void ingot_linear_ws_planes(ingot_linear_ws* ws, void** hi, void** lo) { *hi = ws->hi; *lo = ws->lo; }
cudaError_t ingot_linear_tc_prepared(ingot_linear_ws* ws, int n_in, int n_tok, int planes) {
    if (!act_shape_ok(ws, n_in, n_tok) || !ws->bf16) return cudaErrorInvalidValue;
    ws->planes = planes > 1 ? 2 : 1;
    return set_prepared(ws, n_in, n_tok);
}

// The same with the producer of the activations folded in: rmsnorm(x; norm_w, eps).
cudaError_t ingot_linear_tc_prepare_norm(ingot_linear_ws* ws, const float* x, const float* norm_w, float eps, int n_in, int n_tok,
                                         cudaStream_t s) {
    if (!act_shape_ok(ws, n_in, n_tok) || ws->bf16) return cudaErrorInvalidValue;
    cudaError_t le = launch_pdl(rmsnorm_split_kernel<kActF16Pair>, dim3(n_tok), dim3(256), 0, s, ws->hi, ws->lo, x, norm_w, n_in, n_in, eps);
    if (le != cudaSuccess) return le;
    return set_prepared(ws, n_in, n_tok);
}
cudaError_t ingot_linear_tc_prepare_norm_bf16(ingot_linear_ws* ws, const float* x, const float* norm_w, float eps, int n_in, int n_mean, int n_tok,
                                              int planes, cudaStream_t s) {
    if (!act_shape_ok(ws, n_in, n_tok) || !ws->bf16) return cudaErrorInvalidValue;
    cudaError_t le = planes > 1
        ? launch_pdl(rmsnorm_split_kernel<kActBF16Pair>, dim3(n_tok), dim3(256), 0, s, ws->hi, ws->lo, x, norm_w, n_in, n_mean, eps)
        : launch_pdl(rmsnorm_split_kernel<kActBF16>, dim3(n_tok), dim3(256), 0, s, ws->hi, ws->lo, x, norm_w, n_in, n_mean, eps);
    if (le != cudaSuccess) return le;
    ws->planes = planes > 1 ? 2 : 1;
    return set_prepared(ws, n_in, n_tok);
}

// count <= 3 matrices W_m [n_out_m][n_in] in one launch; matrix m goes to `out` (count == 1, !to_partial) or as k slices to
// scratch slot first_slot + m.
// append: the slices are written behind the ones the slots already hold (all slots of the group must hold the same
// number), so that a second product - the lo plane of a quantised matrix after its hi plane - simply adds k slices
// for the consumer kernel to sum.
// rows_per_block > 0 (count == 1): block-diagonal; n_in is then the row length of one block and the prepared activations hold
// n_out / rows_per_block such blocks side by side.
static cudaError_t launch_gemm(ingot_linear_ws* ws, float* out, const void* const* w, int n_in, const int* n_out, int count,
                               int accumulate, int first_slot, bool to_partial, bool append, cudaStream_t s, int rows_per_block = 0,
                               __half* out_half = nullptr, int half_ld = 0, int half_block = 0) {
    const int n_tok = ws->prepared_tok;
    if (rows_per_block > 0 && (count != 1 || n_out[0] % rows_per_block != 0 || rows_per_block % 4 != 0 || n_in % 8 != 0)) return cudaErrorInvalidValue;
    const int act_in = rows_per_block > 0 ? n_in * (n_out[0] / rows_per_block) : n_in;
    if (act_in != ws->prepared_in || n_tok < 1 || count < 1 || first_slot < 0 || first_slot + count > ws->n_slots || (count > 1 && !to_partial) ||
        (append && !to_partial))
        return cudaErrorInvalidValue;
    const int held = append ? ws->slot_split[first_slot] : 0;
    for (int m = 0; m < count && append; m++)
        if (ws->slot_split[first_slot + m] != held || ws->slot_out[first_slot + m] != n_out[m]) return cudaErrorInvalidValue;
    const CUtensorMap* maps[3] = {nullptr, nullptr, nullptr};
    GemmParams p = {};
    const int tiles_m = (n_tok + kBM - 1) / kBM;
    // 256 outputs per CTA where the operand traffic bounds the kernel (one plane, whole waves of tiles): a 256-wide tile takes
    // about 1.5 times as long as a 128-wide one
    int kBN = 128;
    if (ws->planes == 1 && count == 1 && rows_per_block == 0) {
        const long long waves128 = ((long long)((n_out[0] + 127) / 128) * tiles_m + ws->num_sms - 1) / ws->num_sms;
        const long long waves256 = ((long long)((n_out[0] + 255) / 256) * tiles_m + ws->num_sms - 1) / ws->num_sms;
        if (waves128 > 1 && 3 * waves256 < 2 * waves128) kBN = 256;
        if (const char* e = getenv("INGOT_GEMM_BN")) kBN = atoi(e) == 256 ? 256 : 128;
    }
    int tiles_n = 0, fit = 1 << 30;
    for (int m = 0; m < count; m++) {
        const auto key = std::make_tuple(w[m], n_out[m], n_in, kBN);
        auto it = ws->w_maps.find(key);
        if (it == ws->w_maps.end()) {
            CUtensorMap tm;
            if (!make_map(&tm, w[m], n_out[m], n_in, kBN, ws->bf16)) return cudaErrorUnknown;
            it = ws->w_maps.emplace(key, tm).first;
        }
        maps[m] = &it->second;
        tiles_n += rows_per_block > 0 ? n_out[m] / rows_per_block * ((rows_per_block + kBN - 1) / kBN) : (n_out[m] + kBN - 1) / kBN;
        p.tile_end[m] = tiles_n;
        p.n_out[m] = n_out[m];
        p.partial[m] = ws->partial + (size_t)(first_slot + m) * ws->partial_floats + (size_t)held * n_tok * n_out[m];
        fit = std::min(fit, (int)(ws->partial_floats / ((size_t)n_tok * n_out[m])) - held);
    }
    for (int m = count; m < 3; m++) { maps[m] = maps[count - 1]; p.tile_end[m] = tiles_n; p.n_out[m] = n_out[count - 1]; p.partial[m] = p.partial[count - 1]; }
    const int tiles = tiles_n * tiles_m;
    p.tiles_n = tiles_n;
    p.tiles_m = tiles_m;
    p.a_bytes = ws->box_rows * kBK * 2;
    const int k_steps = (n_in + kBK - 1) / kBK;
    // enough k slices to give every SM a CTA, at least 4 k-steps each, and no more than the slots hold
    if (to_partial && fit < 1) return cudaErrorInvalidValue;
    const int n_split = out_half ? 1 : std::max(1, std::min({ws->num_sms / tiles, k_steps / 4, fit}));
    p.out_half = out_half;
    p.half_ld = half_ld;
    p.half_block = half_block;
    p.out = out; p.status = ws->status;
    p.n_tok = n_tok; p.k_steps = k_steps; p.n_split = n_split; p.accumulate = accumulate;
    p.to_partial = to_partial ? 1 : 0;
    p.idesc = idesc_f16(kBN) | (ws->bf16 ? kIdescBF16 : 0u);
    p.rows_per_block = rows_per_block;
    p.k_block = rows_per_block > 0 ? n_in : 0;
    p.tiles_per_block = rows_per_block > 0 ? (rows_per_block + kBN - 1) / kBN : 0;
    dim3 grid(tiles, 1, n_split);
    auto run = [&](auto kernel, int smem) {
        return launch_pdl(kernel, grid, dim3(kThreads), (size_t)smem, s, ws->map_hi, ws->map_lo, *maps[0], *maps[1], *maps[2], p);
    };
    cudaError_t le = ws->planes > 1 ? run(linear_sm100_kernel<2, 128, false>, Ring<2, 128>::kSmemBytes)
                   : kBN == 256     ? run(linear_sm100_kernel<1, 256, false>, Ring<1, 256>::kSmemBytes)
                                    : run(linear_sm100_kernel<1, 128, false>, Ring<1, 128>::kSmemBytes);
    if (le != cudaSuccess) return le;
    for (int m = 0; m < count; m++) {
        ws->slot_split[first_slot + m] = held + n_split;
        ws->slot_out[first_slot + m] = n_out[m];
    }
    if (!to_partial && n_split > 1) {
        const size_t n = (size_t)n_tok * n_out[0];
        le = launch_pdl(splitk_reduce_kernel, dim3((unsigned)((n / 4 + 255) / 256)), dim3(256), 0, s, out, (const float*)p.partial[0], n_split, n,
                        accumulate);
        if (le != cudaSuccess) return le;
    }
    return cudaGetLastError();
}

// out [n_tok][n_out] (+)= prepared activations x W^T, W f16 [n_out][n_in] on the device.
cudaError_t ingot_linear_tc_run(ingot_linear_ws* ws, float* out, const void* w, int n_in, int n_out, int accumulate, cudaStream_t s) {
    return launch_gemm(ws, out, &w, n_in, &n_out, 1, accumulate, 0, false, false, s);
}

// Block-diagonal product: W [n_out][k_block], output rows of block b = row / rows_per_block times the prepared columns
// b * k_block .. (b + 1) * k_block - 1.
cudaError_t ingot_linear_tc_run_blocks(ingot_linear_ws* ws, float* out, const void* w, int k_block, int n_out, int rows_per_block, cudaStream_t s) {
    return launch_gemm(ws, out, &w, k_block, &n_out, 1, 0, 0, false, false, s, rows_per_block);
}

// Plain (rows_per_block 0) or block-diagonal product with an f16 result: row t at out + t * out_ld, block b's columns from b * out_block
// on. Row lengths and blocks are multiples of 8.
cudaError_t ingot_linear_tc_run_half(ingot_linear_ws* ws, void* out, int out_ld, int out_block, const void* w, int n_in, int n_out, int rows_per_block,
                                     cudaStream_t s) {
    if (out_ld % 8 != 0 || out_block % 8 != 0 || n_out % 8 != 0 || rows_per_block % 8 != 0) return cudaErrorInvalidValue;
    return launch_gemm(ws, nullptr, &w, n_in, &n_out, 1, 0, 0, false, false, s, rows_per_block, static_cast<__half*>(out), out_ld, out_block);
}

// The map of an activation or weight buffer, made once.
static const CUtensorMap* map_of(ingot_linear_ws* ws, const void* base, int rows, int cols, int box, bool bf16) {
    const auto key = std::make_tuple(base, rows, cols, box);
    auto it = ws->w_maps.find(key);
    if (it == ws->w_maps.end()) {
        CUtensorMap tm;
        if (!make_map(&tm, base, rows, cols, box, bf16)) return nullptr;
        it = ws->w_maps.emplace(key, tm).first;
    }
    return &it->second;
}

// out f16 [n_tok][out_ld] = a W^T, both operands f16: a [a_rows][n_in] with n_tok <= a_rows, W [n_out][n_in]. Lengths are multiples of 8.
cudaError_t ingot_linear_tc_run_f16(ingot_linear_ws* ws, void* out, int out_ld, const void* a, int a_rows, int n_tok, const void* w, int n_in, int n_out, cudaStream_t s) {
    if (n_in % 8 != 0 || n_out % 8 != 0 || out_ld % 8 != 0 || n_tok < 1 || n_tok > a_rows) return cudaErrorInvalidValue;
    GemmParams p = {};
    p.tiles_m = (n_tok + kBM - 1) / kBM;
    const long long waves128 = ((long long)((n_out + 127) / 128) * p.tiles_m + ws->num_sms - 1) / ws->num_sms;
    const long long waves256 = ((long long)((n_out + 255) / 256) * p.tiles_m + ws->num_sms - 1) / ws->num_sms;
    const int kBN = waves128 > 1 && 3 * waves256 < 2 * waves128 ? 256 : 128;
    if (ws->w_maps.size() > 65536) ws->w_maps.clear();
    const CUtensorMap *ma = map_of(ws, a, a_rows, n_in, 128, false), *mw = map_of(ws, w, n_out, n_in, kBN, false);
    if (!ma || !mw) return cudaErrorUnknown;
    p.tiles_n = (n_out + kBN - 1) / kBN;
    for (int m = 0; m < 3; m++) { p.n_out[m] = n_out; p.tile_end[m] = p.tiles_n; }
    p.status = ws->status;
    p.n_tok = n_tok;
    p.k_steps = (n_in + kBK - 1) / kBK;
    p.n_split = 1;
    p.a_bytes = kBoxBytes;
    p.idesc = idesc_f16(kBN);
    p.out_half = static_cast<__half*>(out);
    p.half_ld = out_ld;
    auto run = [&](auto kernel, int smem) {
        return launch_pdl(kernel, dim3(p.tiles_n * p.tiles_m), dim3(kThreads), (size_t)smem, s, *ma, *ma, *mw, *mw, *mw, p);
    };
    return kBN == 256 ? run(linear_sm100_kernel<1, 256, false>, Ring<1, 256>::kSmemBytes) : run(linear_sm100_kernel<1, 128, false>, Ring<1, 128>::kSmemBytes);
}

cudaError_t ingot_grouped_tc_run(ingot_linear_ws* ws, const ingot_grouped_gemm* g, cudaStream_t s) {
    if (g->act == 2 && (g->n_out % 64 != 0 || !g->out_hi)) return cudaErrorInvalidValue;
    if (!ws->bf16 || g->n_in % 8 != 0 || g->n_out % 8 != 0 || g->n_rows < 1 || g->n_groups < 1 || g->rows_per_group < 1) return cudaErrorInvalidValue;
    const int planes = g->a_lo ? 2 : 1, box_rows = g->rows_per_group >= 128 ? 128 : (g->rows_per_group + 7) / 8 * 8;
    GemmParams p = {};
    p.tiles_m = g->n_rows / kBM + std::min(g->n_rows, g->n_groups);  // at least as many as there can be
    // as for plain products: 256 outputs per CTA if that saves waves, judged by the row tiles of evenly filled groups
    const int likely = std::max(1, std::min(g->n_groups, g->n_rows) * ((g->n_rows / std::min(g->n_groups, g->n_rows) + kBM - 1) / kBM));
    int kBN = 128;
    if (planes == 1) {
        const long long waves128 = ((long long)((g->n_out + 127) / 128) * likely + ws->num_sms - 1) / ws->num_sms;
        const long long waves256 = ((long long)((g->n_out + 255) / 256) * likely + ws->num_sms - 1) / ws->num_sms;
        if (waves128 > 1 && 3 * waves256 < 2 * waves128) kBN = 256;
    }
    if (ws->w_maps.size() > 65536) ws->w_maps.clear();
    const CUtensorMap* hi = map_of(ws, g->a_hi, g->n_rows, g->n_in, box_rows, true);
    const CUtensorMap* lo = planes > 1 ? map_of(ws, g->a_lo, g->n_rows, g->n_in, box_rows, true) : hi;
    const CUtensorMap* w = map_of(ws, g->w, g->n_groups * g->n_out, g->n_in, kBN, true);
    if (!hi || !lo || !w) return cudaErrorUnknown;
    p.tiles_n = (g->n_out + kBN - 1) / kBN;
    for (int m = 0; m < 3; m++) { p.n_out[m] = g->n_out; p.tile_end[m] = p.tiles_n; }
    p.out = g->out;
    p.status = ws->status;
    p.n_tok = g->n_rows;
    p.k_steps = (g->n_in + kBK - 1) / kBK;
    p.n_split = 1;
    p.a_bytes = box_rows * kBK * 2;
    p.idesc = idesc_f16(kBN) | kIdescBF16;
    p.group_start = g->group_start;
    p.n_groups = g->n_groups;
    p.row_scale = g->row_scale;
    p.act = g->act;
    p.out_hi = static_cast<__nv_bfloat16*>(g->out_hi);
    p.out_lo = static_cast<__nv_bfloat16*>(g->out_lo);
    auto run = [&](auto kernel, int smem) {
        return launch_pdl(kernel, dim3(p.tiles_n * p.tiles_m), dim3(kThreads), (size_t)smem, s, *hi, *lo, *w, *w, *w, p);
    };
    return planes > 1   ? run(linear_sm100_kernel<2, 128, true>, Ring<2, 128>::kSmemBytes)
           : kBN == 256 ? run(linear_sm100_kernel<1, 256, true>, Ring<1, 256>::kSmemBytes)
                        : run(linear_sm100_kernel<1, 128, true>, Ring<1, 128>::kSmemBytes);
}

// The same product left as k slices in scratch slot 0..2 for one of the ingot_linear_tc_finish_* calls below.
cudaError_t ingot_linear_tc_run_partial(ingot_linear_ws* ws, const void* w, int n_in, int n_out, int slot, cudaStream_t s) {
    return launch_gemm(ws, nullptr, &w, n_in, &n_out, 1, 0, slot, true, false, s);
}

// The products of count <= 3 matrices that read the same prepared activations (q/k/v, gate/up), as one launch:
// matrix m is left as k slices in scratch slot m.
// append != 0: the slices are added behind those the slots hold from the call before (same widths).
cudaError_t ingot_linear_tc_run_partial_group(ingot_linear_ws* ws, const void* const* w, int n_in, const int* n_out, int count,
                                              int first_slot, int append, cudaStream_t s) {
    return launch_gemm(ws, nullptr, w, n_in, n_out, count, 0, first_slot, true, append != 0, s);
}

// The product left in `slot`: *n_slices matrices [prepared tokens][n_out] f32 to be summed in order.
const float* ingot_linear_ws_slices(const ingot_linear_ws* ws, int slot, int* n_slices) {
    *n_slices = ws->slot_split[slot];
    return ws->partial + (size_t)slot * ws->partial_floats;
}

static Slices slices_of(const ingot_linear_ws* ws, int slot) {
    return Slices{ws->partial + (size_t)slot * ws->partial_floats, ws->slot_split[slot]};
}

// outs[m] = product left in slot m, for count <= 3 outputs (q, k, v) in one launch.
cudaError_t ingot_linear_tc_finish_group(ingot_linear_ws* ws, float* const* outs, int count, cudaStream_t s) {
    if (count < 1 || count > 3) return cudaErrorInvalidValue;
    FinishGroup g = {};
    int widest = 0;
    for (int m = 0; m < count; m++) {
        g.in[m] = slices_of(ws, m);
        g.out[m] = outs[m];
        g.n_out[m] = ws->slot_out[m];
        widest = std::max(widest, ws->slot_out[m]);
    }
    const size_t n = (size_t)ws->prepared_tok * widest;
    cudaError_t le = launch_pdl(finish_group_kernel, dim3((unsigned)((n / 4 + 255) / 256), count), dim3(256), 0, s, g, ws->prepared_tok);
    if (le != cudaSuccess) return le;
    return cudaGetLastError();
}

// x += product left in `slot` (the residual add), then, with norm_w, the hi/lo activations of rmsnorm(x; norm_w, eps)
// become the prepared input of the next projections (n_in = the product's width).
cudaError_t ingot_linear_tc_finish_residual_norm(ingot_linear_ws* ws, float* x, const float* norm_w, float eps, int slot, cudaStream_t s) {
    const int n = ws->slot_out[slot], n_tok = ws->prepared_tok;
    if (n % 4 != 0 || (norm_w && !act_shape_ok(ws, n, n_tok)) || ws->bf16) return cudaErrorInvalidValue;
    cudaError_t le = launch_pdl(finish_residual_norm_kernel<kActF16Pair>, dim3(n_tok), dim3(256), 0, s, x, slices_of(ws, slot), ws->hi, ws->lo, norm_w, n, n, n_tok, eps, (const float*)nullptr, (const int32_t*)nullptr, 0);
    if (le != cudaSuccess) return le;
    return norm_w ? set_prepared(ws, n, n_tok) : cudaGetLastError();
}
// pair_rows (null: none): x[t] also takes in the rows row_of[t * top + k] of it.
cudaError_t ingot_linear_tc_finish_residual_norm_bf16(ingot_linear_ws* ws, float* x, const float* norm_w, float eps, int n_mean, int planes,
                                                      const float* pair_rows, const int32_t* row_of, int top, cudaStream_t s) {
    if (!pair_rows) top = 0;
    const int n = ws->slot_out[0], n_tok = ws->prepared_tok;
    if (n % 4 != 0 || (norm_w && !act_shape_ok(ws, n, n_tok)) || !ws->bf16) return cudaErrorInvalidValue;
    cudaError_t le = planes > 1
        ? launch_pdl(finish_residual_norm_kernel<kActBF16Pair>, dim3(n_tok), dim3(256), 0, s, x, slices_of(ws, 0), ws->hi, ws->lo, norm_w, n, n_mean, n_tok, eps, pair_rows, row_of, top)
        : launch_pdl(finish_residual_norm_kernel<kActBF16>, dim3(n_tok), dim3(256), 0, s, x, slices_of(ws, 0), ws->hi, ws->lo, norm_w, n, n_mean, n_tok, eps, pair_rows, row_of, top);
    if (le != cudaSuccess) return le;
    ws->planes = planes > 1 ? 2 : 1;
    return norm_w ? set_prepared(ws, n, n_tok) : cudaGetLastError();
}

// The product in slot 0 (width 2 n: gate half, up half) becomes the bf16 operand act(gate) * up of the next product.
cudaError_t ingot_linear_tc_finish_gated_bf16(ingot_linear_ws* ws, int act, int planes, cudaStream_t s) {
    const int n = ws->slot_out[0] / 2, n_tok = ws->prepared_tok;
    if (!ws->bf16 || n % 8 != 0 || !act_shape_ok(ws, n, n_tok)) return cudaErrorInvalidValue;
    const dim3 grid((unsigned)((n / 4 + 255) / 256), n_tok);
    cudaError_t le = planes > 1
        ? launch_pdl(finish_gated_kernel<kActBF16Pair>, grid, dim3(256), 0, s, ws->hi, ws->lo, slices_of(ws, 0), n, (size_t)n_tok * 2 * n, act)
        : launch_pdl(finish_gated_kernel<kActBF16>, grid, dim3(256), 0, s, ws->hi, ws->lo, slices_of(ws, 0), n, (size_t)n_tok * 2 * n, act);
    if (le != cudaSuccess) return le;
    ws->planes = planes > 1 ? 2 : 1;
    return set_prepared(ws, n, n_tok);
}

// hi/lo of silu(slot_gate) .* slot_up become the prepared input of the next projection.
cudaError_t ingot_linear_tc_finish_swiglu(ingot_linear_ws* ws, int slot_gate, int slot_up, cudaStream_t s) {
    const int n_in = ws->slot_out[slot_gate], n_tok = ws->prepared_tok;
    const size_t n = (size_t)n_tok * n_in;
    if (ws->slot_out[slot_up] != n_in || n > ws->act_elems || n_in % kBK != 0) return cudaErrorInvalidValue;
    cudaError_t le = launch_pdl(finish_swiglu_kernel, dim3((unsigned)((n / 4 + 255) / 256)), dim3(256), 0, s, ws->hi, ws->lo, slices_of(ws, slot_gate), slices_of(ws, slot_up), n);
    if (le != cudaSuccess) return le;
    return set_prepared(ws, n_in, n_tok);
}

int* ingot_linear_ws_status_dev(ingot_linear_ws* ws) { return ws->status; }

// The status word: non-zero after a bounded wait expired in some launch since the last call. Synchronises the device.
int ingot_linear_ws_status(ingot_linear_ws* ws) {
    int v = 0;
    if (cudaMemcpy(&v, ws->status, sizeof(int), cudaMemcpyDeviceToHost) != cudaSuccess) return -1;
    if (v) cudaMemset(ws->status, 0, sizeof(int));
    return v;
}

}  // extern "C"
