// Support kernels for CudaBackend: the non-attention stages of the forward pass
// (src/cpu_backend.cpp:39-42, 71-85; Metal: rmsnorm / matvec_f16 / silu_mul,
// shaders/kernels.metal:129-252, 706-710). Activations stay f32 everywhere, weights are read in their
// stored type (f16 or f32) and widened, products accumulate in f32 — the arithmetic of ops::dot_row
// (src/ops.cpp:127-141) up to summation order — so that greedy decoding follows the CPU reference.
// bf16 weights (models loaded from safetensors folders) are read the same way: widened, never rounded further.
// Single-token steps with f16 weights use the weight-streaming kernel (gemv_stream_kernel); batches use the
// tensor-core kernel of linear_sm100.cu; the plain kernels here cover f32 weights and odd shapes.
#include <algorithm>
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <type_traits>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdlib.h>

// Longest input row the weight-streaming GEMV stages in shared memory: n_in floats plus a few words of static
// shared memory must stay inside the 48 KB a kernel gets without an opt-in.
constexpr int kGemvMaxIn = 12032;

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// out[row][i] = x[row][i] * rsqrt(mean(x[row]^2) + eps) * w[i]      (ops::rmsnorm, src/ops.cpp:227-232)
__global__ void rmsnorm_kernel(float* out, const float* x, const float* w, int n, float eps) {
    __shared__ float red[32];
    const float* xr = x + (size_t)blockIdx.x * n;
    float* orow = out + (size_t)blockIdx.x * n;
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) ss += xr[i] * xr[i];
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    if (threadIdx.x < 32) {
        float v = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0.f;
        v = warp_sum(v);
        if (threadIdx.x == 0) red[0] = 1.0f / sqrtf(v / float(n) + eps);
    }
    __syncthreads();
    const float scale = red[0];
    for (int i = threadIdx.x; i < n; i += blockDim.x) orow[i] = xr[i] * scale * w[i];
}

// The same with a row gather, and with the mean over n_mean of the row's n floats (rows zero-padded to an aligned length).
__global__ void rmsnorm_rows_kernel(float* out, const float* x, const float* w, const int32_t* rows, int n, int n_mean, float eps) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
    __shared__ float red[32];
    const float* xr = x + (size_t)(rows ? rows[blockIdx.x] : (int)blockIdx.x) * n;
    float* orow = out + (size_t)blockIdx.x * n;
    constexpr int kKeep = 8;  // float4s of the row a thread keeps between the two passes
    const int n4 = n % 4 == 0 ? n / 4 : 0;
    float4 v[kKeep];
    float ss = 0.f;
    if (n4) {
#pragma unroll
        for (int k = 0; k < kKeep; k++) {
            const int i = threadIdx.x + k * blockDim.x;
            v[k] = i < n4 ? reinterpret_cast<const float4*>(xr)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int k = 0; k < kKeep; k++) { ss += v[k].x * v[k].x; ss += v[k].y * v[k].y; ss += v[k].z * v[k].z; ss += v[k].w * v[k].w; }
    }
    const int kept = n4 ? min(n, kKeep * 4 * (int)blockDim.x) : 0;
    for (int i = kept + threadIdx.x; i < n; i += blockDim.x) ss += xr[i] * xr[i];
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < (int)(blockDim.x >> 5); i++) t += red[i];
    const float scale = 1.0f / sqrtf(t / float(n_mean) + eps);
    if (n4) {
#pragma unroll
        for (int k = 0; k < kKeep; k++) {
            const int i = threadIdx.x + k * blockDim.x;
            if (i >= n4) break;
            const float4 g = reinterpret_cast<const float4*>(w)[i];
            reinterpret_cast<float4*>(orow)[i] = make_float4(v[k].x * scale * g.x, v[k].y * scale * g.y, v[k].z * scale * g.z, v[k].w * scale * g.w);
        }
    }
    for (int i = kept + threadIdx.x; i < n; i += blockDim.x) orow[i] = xr[i] * scale * w[i];
}

// Activation of gated feed-forwards: 0 silu, 1 the tanh form of gelu.
__device__ __forceinline__ float gate_act(float g, int act) {
    if (act == 0) return g / (1.0f + expf(-g));
    return 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
}
__global__ void gated_act_kernel(float* out, const float* in, int n, size_t total, int act) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const size_t r = i / n, c = i - r * n;
    out[i] = gate_act(in[r * 2 * n + c], act) * in[r * 2 * n + n + c];
}

// gate[i] = silu(gate[i]) * up[i]      (src/cpu_backend.cpp:79, ops::silu src/ops.h:35)
__global__ void silu_mul_kernel(float* gate, const float* up, size_t n) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) {
        const float g = gate[i];
        gate[i] = g / (1.0f + expf(-g)) * up[i];
    }
}

template <typename W>
__device__ __forceinline__ void load8(const W* p, float (&w)[8]);
template <>
__device__ __forceinline__ void load8<__half>(const __half* p, float (&w)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __half2* h = reinterpret_cast<const __half2*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const float2 f = __half22float2(h[i]);
        w[2 * i] = f.x;
        w[2 * i + 1] = f.y;
    }
}
template <>
__device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&w)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const uint32_t u[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {  // a bf16 value is the high half of the f32 with the same bits
        w[2 * i] = __uint_as_float(u[i] << 16);
        w[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
    }
}
template <>
__device__ __forceinline__ void load8<float>(const float* p, float (&w)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    w[0] = a.x; w[1] = a.y; w[2] = a.z; w[3] = a.w; w[4] = b.x; w[5] = b.y; w[6] = b.z; w[7] = b.w;
}

// Activation rows may be longer than n_in (x_ld apart), and the matrix may be block-diagonal: with rows_per_block > 0,
// output row r reads the n_in columns that start at (r / rows_per_block) * n_in.
struct XLayout {
    int ld, rows_per_block;
    __device__ __forceinline__ int col0(int row, int n_in) const { return rows_per_block > 0 ? (row / rows_per_block) * n_in : 0; }
};

// out[t][r] (+)= dot(W[r][:], x[t][:]) for a tile of TT tokens; one warp per output row.
// W is [n_out][n_in] row-major (ggml ne = [n_in, n_out]); n_in is a multiple of 8.
template <typename W, int TT>
__global__ void linear_kernel(float* out, const W* w, const float* x, int n_in, int n_out, int n_tok, int accumulate, XLayout xl) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    const int t0 = blockIdx.y * TT;
    if (row >= n_out) return;
    const W* wr = w + (size_t)row * n_in;
    const float* x0 = x + xl.col0(row, n_in);
    float acc[TT];
#pragma unroll
    for (int t = 0; t < TT; t++) acc[t] = 0.f;
    for (int i = lane * 8; i < n_in; i += 256) {
        float wv[8];
        load8<W>(wr + i, wv);
#pragma unroll
        for (int t = 0; t < TT; t++) {
            if (t0 + t < n_tok) {
                const float* xr = x0 + (size_t)(t0 + t) * xl.ld + i;
                const float4 a = *reinterpret_cast<const float4*>(xr), b = *reinterpret_cast<const float4*>(xr + 4);
                acc[t] = fmaf(wv[0], a.x, acc[t]); acc[t] = fmaf(wv[1], a.y, acc[t]);
                acc[t] = fmaf(wv[2], a.z, acc[t]); acc[t] = fmaf(wv[3], a.w, acc[t]);
                acc[t] = fmaf(wv[4], b.x, acc[t]); acc[t] = fmaf(wv[5], b.y, acc[t]);
                acc[t] = fmaf(wv[6], b.z, acc[t]); acc[t] = fmaf(wv[7], b.w, acc[t]);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < TT; t++) {
        const float v = warp_sum(acc[t]);
        if (lane == 0 && t0 + t < n_tok) {
            float* o = out + (size_t)(t0 + t) * n_out + row;
            *o = accumulate ? *o + v : v;
        }
    }
}


// Single-token form (decode): HBM-bound streaming of the weight matrix. One warp per output row; each lane
// keeps four 16-byte weight loads in flight (2 KB per warp, up to 128 KB per SM) and reads x through L1.
// out[r] (+)= dot(W[r][:], x).
template <typename W>
__global__ void __launch_bounds__(256) gemv_kernel(float* out, const W* w, const float* x, int n_in, int n_out, int accumulate) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row = blockIdx.x * (blockDim.x >> 5) + warp;
    if (row >= n_out) return;
    const W* wr = w + (size_t)row * n_in;
    float acc0 = 0.f, acc1 = 0.f, acc2 = 0.f, acc3 = 0.f;
    auto fma8 = [&](float& acc, const float (&wv)[8], const float* xs) {
        const float4 xa = *reinterpret_cast<const float4*>(xs), xb = *reinterpret_cast<const float4*>(xs + 4);
        acc = fmaf(wv[0], xa.x, acc); acc = fmaf(wv[1], xa.y, acc); acc = fmaf(wv[2], xa.z, acc); acc = fmaf(wv[3], xa.w, acc);
        acc = fmaf(wv[4], xb.x, acc); acc = fmaf(wv[5], xb.y, acc); acc = fmaf(wv[6], xb.z, acc); acc = fmaf(wv[7], xb.w, acc);
    };
    int i = lane * 8;
    for (; i + 768 < n_in; i += 1024) {
        float p0[8], p1[8], p2[8], p3[8];
        load8<W>(wr + i, p0); load8<W>(wr + i + 256, p1); load8<W>(wr + i + 512, p2); load8<W>(wr + i + 768, p3);
        fma8(acc0, p0, x + i); fma8(acc1, p1, x + i + 256); fma8(acc2, p2, x + i + 512); fma8(acc3, p3, x + i + 768);
    }
    for (; i < n_in; i += 256) {
        float p0[8];
        load8<W>(wr + i, p0);
        fma8(acc0, p0, x + i);
    }
    const float v = warp_sum((acc0 + acc1) + (acc2 + acc3));
    if (lane == 0) out[row] = accumulate ? out[row] + v : v;
}

// Few long rows: one CTA per row, all of whose threads request their share of the row (up to four loads each) before the wait
// for the preceding kernel. A warp per row would leave most SMs without work.
__global__ void __launch_bounds__(256) gemv_row_kernel(float* out, const __nv_bfloat16* w, const float* x, int n_in, int accumulate) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    __shared__ float red[8];
    const __nv_bfloat16* wr = w + (size_t)blockIdx.x * n_in;
    const int i0 = threadIdx.x * 8;
    float p[4][8];
#pragma unroll
    for (int j = 0; j < 4; j++)
        if (i0 + j * 2048 < n_in) load8<__nv_bfloat16>(wr + i0 + j * 2048, p[j]);
    asm volatile("griddepcontrol.wait;" ::: "memory");
    float acc = 0.f;
    auto fma8 = [&](const float (&v)[8], const float* xs) {
        const float4 a = *reinterpret_cast<const float4*>(xs), b = *reinterpret_cast<const float4*>(xs + 4);
        acc = fmaf(v[0], a.x, acc); acc = fmaf(v[1], a.y, acc); acc = fmaf(v[2], a.z, acc); acc = fmaf(v[3], a.w, acc);
        acc = fmaf(v[4], b.x, acc); acc = fmaf(v[5], b.y, acc); acc = fmaf(v[6], b.z, acc); acc = fmaf(v[7], b.w, acc);
    };
#pragma unroll
    for (int j = 0; j < 4; j++)
        if (i0 + j * 2048 < n_in) fma8(p[j], x + i0 + j * 2048);
    for (int i = i0 + 8192; i < n_in; i += 2048) {
        float v[8];
        load8<__nv_bfloat16>(wr + i, v);
        fma8(v, x + i);
    }
    acc = warp_sum(acc);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = acc;
    __syncthreads();
    if (threadIdx.x == 0) {
        float t = 0.f;
        for (int i = 0; i < 8; i++) t += red[i];
        out[blockIdx.x] = accumulate ? out[blockIdx.x] + t : t;
    }
}

// Single-token products with f16 weights: a weight-streaming kernel, HBM-bound by design.
//   out_m[r] (+)= dot(W_m[r][:], x')            x' = x, or x .* norm_w with the result scaled by
//   rsqrt(mean(x^2) + eps) (the RMS norm of ops::rmsnorm, src/ops.cpp:227-232, folded in; the same product up to
//   rounding order), for up to three matrices that read the same vector (q/k/v), or for the gate/up pair with
//   out[r] = silu(gate[r]) * up[r] as the epilogue (src/cpu_backend.cpp:79).
// One launch is one resident wave of CTAs; a warp owns whole rows (r, r + W, ...), W chosen so that all warps get
// the same number of rows. A lane keeps four (or six) 16-byte weight loads in flight and requests the next set before
// it consumes the current ones, across row boundaries too, so a warp streams without gaps. x' is staged in
// shared memory once per CTA. Under programmatic dependent launch the first weight loads are issued before
// the wait for the preceding kernel (weights never depend on it), which hides the ramp of every launch
// behind the tail of the previous one.
struct GemvGroup {
    const void* w[3];      // weight rows: f16 values, or the quant plane of a repacked Q8_0 / Q4_0 matrix
    const __half* d[3];    // block scales of a quantised matrix (one per 32 weights), else null
    float* out[3];
    int row_end[3];  // running totals of the matrices' row counts
    int n_mat;
};

__device__ __forceinline__ uint4 ld_stream_u4(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
// x' is staged in shared memory in the order the lanes consume it: the j-th float4 that lane l needs for a chunk
// sits at float4 index (chunk * J + j) * 32 + l (J = float4s per lane and chunk), so that the 32 lanes of a warp
// read 32 consecutive float4s - conflict-free - instead of 32 segments that are 32 to 128 bytes apart (a 2- to 8-way
// bank conflict on every read, which cost more shared-memory cycles than the weights cost HBM cycles).
__device__ __forceinline__ float dot8(const uint4& raw, const float4* x4) {
    const __half2* h = reinterpret_cast<const __half2*>(&raw);
    const float4 xa = x4[0], xb = x4[32];
    const float2 w0 = __half22float2(h[0]), w1 = __half22float2(h[1]), w2 = __half22float2(h[2]), w3 = __half22float2(h[3]);
    float acc = w0.x * xa.x;
    acc = fmaf(w0.y, xa.y, acc); acc = fmaf(w1.x, xa.z, acc); acc = fmaf(w1.y, xa.w, acc);
    acc = fmaf(w2.x, xb.x, acc); acc = fmaf(w2.y, xb.y, acc); acc = fmaf(w3.x, xb.z, acc); acc = fmaf(w3.y, xb.w, acc);
    return acc;
}

__device__ __forceinline__ float dot8_bf16(const uint4& raw, const float4* x4) {
    const float4 xa = x4[0], xb = x4[32];
    float acc = __uint_as_float(raw.x << 16) * xa.x;
    acc = fmaf(__uint_as_float(raw.x & 0xffff0000u), xa.y, acc);
    acc = fmaf(__uint_as_float(raw.y << 16), xa.z, acc); acc = fmaf(__uint_as_float(raw.y & 0xffff0000u), xa.w, acc);
    acc = fmaf(__uint_as_float(raw.z << 16), xb.x, acc); acc = fmaf(__uint_as_float(raw.z & 0xffff0000u), xb.y, acc);
    acc = fmaf(__uint_as_float(raw.w << 16), xb.z, acc); acc = fmaf(__uint_as_float(raw.w & 0xffff0000u), xb.w, acc);
    return acc;
}

// Weight formats of the streaming kernel. A lane's 16-byte load covers kElems weights: 8 f16 values, 16 Q8_0
// quants (half a block) or the 32 nibbles of one Q4_0 block; the 32 lanes of a warp therefore cover 512 bytes =
// 256 / 512 / 1024 consecutive weights per load. Quantised rows come from the repacked planes of
// quant_kernels.cu: quants contiguous per row, one f16 scale per 32 weights in a plane of its own.
enum : int { kFmtF16 = 0, kFmtQ8_0 = 1, kFmtQ4_0 = 2, kFmtBF16 = 3 };
template <int kFmt> struct FmtTraits {
    static constexpr int kElems = kFmt == kFmtQ8_0 ? 16 : kFmt == kFmtQ4_0 ? 32 : 8;
    static constexpr bool kPlain = kFmt == kFmtF16 || kFmt == kFmtBF16;  // no block scales
};

__device__ __forceinline__ uint32_t prmt_b(uint32_t a, uint32_t b, uint32_t sel) {
    uint32_t r;
    asm("prmt.b32 %0, %1, %2, %3;" : "=r"(r) : "r"(a), "r"(b), "r"(sel));
    return r;
}
// byte k of `word` as a float: the byte becomes the low mantissa bits of 2^23, then 2^23 + bias is subtracted
__device__ __forceinline__ float byte_f(uint32_t word, int k, float bias) {
    return __uint_as_float(prmt_b(word, 0x4B000000u, 0x7650u + (uint32_t)k)) - bias;
}
// d * sum_i q_i x_i over the weights of one 16-byte load (the grouping of dot_q8_0 / dot_q4_0, src/ops.cpp:143-180)
template <int kFmt>
__device__ __forceinline__ float dot_load(const uint4& raw, const float4* x4, unsigned short scale_bits) {
    if (kFmt == kFmtF16) return dot8(raw, x4);
    if (kFmt == kFmtBF16) return dot8_bf16(raw, x4);
    const float d = __half2float(__ushort_as_half(scale_bits));
    const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
    float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
    if (kFmt == kFmtQ8_0) {
#pragma unroll
        for (int j = 0; j < 4; j++) {  // signed byte = (byte ^ 0x80) - 128
            const uint32_t u = w[j] ^ 0x80808080u;
            const float4 xv = x4[j * 32];
            s0 = fmaf(byte_f(u, 0, 8388608.f + 128.f), xv.x, s0);
            s1 = fmaf(byte_f(u, 1, 8388608.f + 128.f), xv.y, s1);
            s2 = fmaf(byte_f(u, 2, 8388608.f + 128.f), xv.z, s2);
            s3 = fmaf(byte_f(u, 3, 8388608.f + 128.f), xv.w, s3);
        }
    } else {
#pragma unroll
        for (int j = 0; j < 4; j++) {  // bytes 4j..4j+3: low nibbles are weights 4j.., high nibbles weights 16+4j..
            const uint32_t lo = w[j] & 0x0F0F0F0Fu, hi = (w[j] >> 4) & 0x0F0F0F0Fu;
            const float4 xl = x4[j * 32];
            const float4 xh = x4[(4 + j) * 32];
            s0 = fmaf(byte_f(lo, 0, 8388608.f + 8.f), xl.x, s0);
            s1 = fmaf(byte_f(lo, 1, 8388608.f + 8.f), xl.y, s1);
            s2 = fmaf(byte_f(lo, 2, 8388608.f + 8.f), xl.z, s2);
            s3 = fmaf(byte_f(lo, 3, 8388608.f + 8.f), xl.w, s3);
            s0 = fmaf(byte_f(hi, 0, 8388608.f + 8.f), xh.x, s0);
            s1 = fmaf(byte_f(hi, 1, 8388608.f + 8.f), xh.y, s1);
            s2 = fmaf(byte_f(hi, 2, 8388608.f + 8.f), xh.z, s2);
            s3 = fmaf(byte_f(hi, 3, 8388608.f + 8.f), xh.w, s3);
        }
    }
    return ((s0 + s1) + (s2 + s3)) * d;
}

// kLoads: 16-byte weight loads per lane and step (split between gate and up under kSwiGLU). Current and next step
// are in flight together, so with kLoads = 6 a whole row of 3072 weights (12 chunks) is requested at once.
// Threads per CTA: every CTA stages x' (and reads the norm weights) for itself, so fewer, larger CTAs mean less of that
// L2 traffic per launch. f16 rows need 80 registers per thread and fit 768 threads (24 warps, one CTA per SM);
// the quantised formats need up to 122 and stay at 256 threads, two or three CTAs per SM (512-thread CTAs measured:
// Q8_0 tg32 561 -> 536 tok/s, Q4_0 539 -> 544).
template <int kFmt>
struct StreamThreads { static constexpr int value = FmtTraits<kFmt>::kPlain ? 768 : 256; };

template <bool kNorm, bool kSwiGLU, int kLoads, int kFmt>
__global__ void __launch_bounds__(StreamThreads<kFmt>::value) gemv_stream_kernel(const GemvGroup g, const float* x, const float* norm_w, float eps, int n_in,
                                                          int total_rows, int accumulate, int use_pdl, int n_mean, int act) {
    extern __shared__ float xs[];  // x', n_in floats
    __shared__ float red[25];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // Rows go round-robin over all warps of the grid, warp-major (warp w of CTA b is number w * gridDim.x + b): when the
    // rows do not divide by the warp count, the warps with one row more are the low-numbered warps of EVERY CTA, so
    // every SM streams the same number of bytes.
    const int W = gridDim.x * (blockDim.x >> 5), gw = warp * gridDim.x + blockIdx.x;
    if (use_pdl) asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    constexpr int kPer = kSwiGLU ? kLoads / 2 : kLoads;  // 512-byte chunks per matrix and step
    constexpr int kElems = FmtTraits<kFmt>::kElems;       // weights per lane and load
    const int n_chunks = n_in / (32 * kElems);
    const int steps = (n_chunks + kPer - 1) / kPer;
    const size_t row_bytes = (size_t)n_chunks * 512;
    const int row_scales = n_in >> 5;

    auto row_base = [&](int r, const char*& wa, const char*& wb, const __half*& da, const __half*& db) {
        if (kSwiGLU) {
            wa = static_cast<const char*>(g.w[0]) + (size_t)r * row_bytes;
            wb = static_cast<const char*>(g.w[1]) + (size_t)r * row_bytes;
            da = FmtTraits<kFmt>::kPlain ? nullptr : g.d[0] + (size_t)r * row_scales;
            db = FmtTraits<kFmt>::kPlain ? nullptr : g.d[1] + (size_t)r * row_scales;
        } else {
            const int m = (r >= g.row_end[0]) + (r >= g.row_end[1] && g.n_mat > 2);
            const int local = m == 0 ? r : r - (m == 1 ? g.row_end[0] : g.row_end[1]);
            wa = static_cast<const char*>(m == 0 ? g.w[0] : m == 1 ? g.w[1] : g.w[2]) + (size_t)local * row_bytes;
            da = FmtTraits<kFmt>::kPlain ? nullptr : (m == 0 ? g.d[0] : m == 1 ? g.d[1] : g.d[2]) + (size_t)local * row_scales;
            wb = nullptr;
            db = nullptr;
        }
    };
    // SA / SB: the block scale that goes with each load (quantised formats)
    auto issue = [&](uint4 (&A)[kPer], uint4 (&B)[kPer], unsigned short (&SA)[kPer], unsigned short (&SB)[kPer], int r, int st) {
        const char *wa, *wb;
        const __half *da, *db;
        row_base(r, wa, wb, da, db);
#pragma unroll
        for (int h = 0; h < kPer; h++) {
            const int c = st * kPer + h;
            if (c < n_chunks) {
                A[h] = ld_stream_u4(wa + (size_t)c * 512 + lane * 16);
                if (kSwiGLU) B[h] = ld_stream_u4(wb + (size_t)c * 512 + lane * 16);
                if (!FmtTraits<kFmt>::kPlain) {
                    const int blk = ((c * 32 + lane) * kElems) >> 5;
                    SA[h] = __ldg(reinterpret_cast<const unsigned short*>(da) + blk);
                    if (kSwiGLU) SB[h] = __ldg(reinterpret_cast<const unsigned short*>(db) + blk);
                }
            }
        }
    };

    uint4 cur_a[kPer], cur_b[kPer], nxt_a[kPer], nxt_b[kPer];
    unsigned short cs_a[kPer] = {}, cs_b[kPer] = {}, ns_a[kPer] = {}, ns_b[kPer] = {};
    int r = gw, st = 0;
    bool have = r < total_rows;
    if (have) issue(cur_a, cur_b, cs_a, cs_b, r, 0);  // before the wait below: weights do not depend on the preceding kernel

    if (use_pdl) asm volatile("griddepcontrol.wait;" ::: "memory");
    float ss = 0.f;
    for (int i = threadIdx.x * 4; i < n_in; i += blockDim.x * 4) {
        float4 v = *reinterpret_cast<const float4*>(x + i);
        if (kNorm) {
            ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
            const float4 n = *reinterpret_cast<const float4*>(norm_w + i);
            v.x *= n.x; v.y *= n.y; v.z *= n.z; v.w *= n.w;
        }
        // element i = chunk * 32 * kElems + lane * kElems + 4 j + t  ->  float4 index (chunk * J + j) * 32 + lane
        const int chunk_e = 32 * kElems, c = i / chunk_e, rem = i - c * chunk_e, l = rem / kElems, jj = (rem - l * kElems) >> 2;
        reinterpret_cast<float4*>(xs)[(c * (kElems / 4) + jj) * 32 + l] = v;
    }
    if (kNorm) {
        ss = warp_sum(ss);
        if (lane == 0) red[warp] = ss;
    }
    __syncthreads();
    float scale = 1.0f;
    if (kNorm) {
        float t = 0.f;
        for (int w = 0; w < (int)(blockDim.x >> 5); w++) t += red[w];
        scale = 1.0f / sqrtf(t / float(n_mean) + eps);
    }

    float acc_a = 0.f, acc_b = 0.f;
    while (have) {
        int r2 = r, st2 = st + 1;
        if (st2 == steps) { st2 = 0; r2 = r + W; }
        const bool have2 = r2 < total_rows;
        if (have2) issue(nxt_a, nxt_b, ns_a, ns_b, r2, st2);
#pragma unroll
        for (int h = 0; h < kPer; h++) {
            const int c = st * kPer + h;
            if (c < n_chunks) {
                const float4* xp = reinterpret_cast<const float4*>(xs) + c * (kElems / 4) * 32 + lane;
                acc_a += dot_load<kFmt>(cur_a[h], xp, cs_a[h]);
                if (kSwiGLU) acc_b += dot_load<kFmt>(cur_b[h], xp, cs_b[h]);
            }
        }
        if (st == steps - 1) {
            acc_a = warp_sum(acc_a);
            if (kSwiGLU) acc_b = warp_sum(acc_b);
            if (lane == 0) {
                if (kSwiGLU) {
                    const float gt = acc_a * scale, up = acc_b * scale;
                    g.out[0][r] = gate_act(gt, act) * up;
                } else {
                    const int m = (r >= g.row_end[0]) + (r >= g.row_end[1] && g.n_mat > 2);
                    const int local = m == 0 ? r : r - (m == 1 ? g.row_end[0] : g.row_end[1]);
                    float* o = (m == 0 ? g.out[0] : m == 1 ? g.out[1] : g.out[2]) + local;
                    const float v = acc_a * scale;
                    *o = accumulate ? *o + v : v;
                }
            }
            acc_a = 0.f;
            acc_b = 0.f;
        }
#pragma unroll
        for (int h = 0; h < kPer; h++) { cur_a[h] = nxt_a[h]; cs_a[h] = ns_a[h]; if (kSwiGLU) { cur_b[h] = nxt_b[h]; cs_b[h] = ns_b[h]; } }
        r = r2; st = st2; have = have2;
    }
}

// Batched form (prefill): out[t][r] (+)= dot(W[r][:], x[t][:]) as a shared-memory tiled f32 GEMM on the FMA
// pipes: 128 tokens x 64 outputs per CTA, k-steps of 16, 8x4 outputs per thread; weights are widened to
// f32 when they are staged. The whole token batch of a prefill chunk up to 128 sits in one tile, so the
// weight matrix is read once per 128 tokens.
constexpr int kGM = 128, kGN = 64, kGK = 16;
template <typename W>
__global__ void __launch_bounds__(256) gemm_kernel(float* out, const W* w, const float* x, int n_in, int n_out, int n_tok, int accumulate, XLayout xl) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
    __shared__ __align__(16) float xs[kGK][kGM + 4];
    __shared__ __align__(16) float ws[kGK][kGN + 4];
    const int t0 = blockIdx.y * kGM;
    // block-diagonal matrices: the output tiles of a block never straddle into the next one
    const int tiles_per_block = xl.rows_per_block > 0 ? (xl.rows_per_block + kGN - 1) / kGN : 0;
    const int blk = tiles_per_block ? blockIdx.x / tiles_per_block : 0;
    const int r0 = tiles_per_block ? blk * xl.rows_per_block + (blockIdx.x - blk * tiles_per_block) * kGN : blockIdx.x * kGN;
    const int r_end = tiles_per_block ? (blk + 1) * xl.rows_per_block : n_out;
    const float* x0 = x + (tiles_per_block ? blk * n_in : 0);
    const int tid = threadIdx.x;
    const int tm = (tid >> 4) * 8, tn = (tid & 15) * 4;  // this thread's 8 tokens x 4 outputs
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    // staging assignments: x tile 128 x 16 floats = 512 float4 (2 per thread); w tile 64 x 16 = 128 chunks of 8 (threads 0..127)
    for (int k0 = 0; k0 < n_in; k0 += kGK) {
#pragma unroll
        for (int it = 0; it < 2; it++) {
            const int idx = it * 256 + tid;
            const int row = idx >> 2, c4 = (idx & 3) * 4;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (t0 + row < n_tok && k0 + c4 < n_in) v = *reinterpret_cast<const float4*>(x0 + (size_t)(t0 + row) * xl.ld + k0 + c4);
            xs[c4 + 0][row] = v.x; xs[c4 + 1][row] = v.y; xs[c4 + 2][row] = v.z; xs[c4 + 3][row] = v.w;
        }
        if (tid < 128) {
            const int row = tid >> 1, c8 = (tid & 1) * 8;
            float wv[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            if (r0 + row < r_end && k0 + c8 < n_in) load8<W>(w + (size_t)(r0 + row) * n_in + k0 + c8, wv);
#pragma unroll
            for (int i = 0; i < 8; i++) ws[c8 + i][row] = wv[i];
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kGK; k++) {
            const float4 xa = *reinterpret_cast<const float4*>(&xs[k][tm]), xb = *reinterpret_cast<const float4*>(&xs[k][tm + 4]);
            const float4 wv = *reinterpret_cast<const float4*>(&ws[k][tn]);
            const float xv[8] = {xa.x, xa.y, xa.z, xa.w, xb.x, xb.y, xb.z, xb.w};
            const float wq[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
            for (int i = 0; i < 8; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(xv[i], wq[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const int t = t0 + tm + i;
        if (t >= n_tok) continue;
        float* o = out + (size_t)t * n_out + r0 + tn;
        if (r0 + tn + 3 < r_end) {
            float4 v = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
            if (accumulate) {
                const float4 old = *reinterpret_cast<const float4*>(o);
                v.x += old.x; v.y += old.y; v.z += old.z; v.w += old.w;
            }
            *reinterpret_cast<float4*>(o) = v;
        } else {
            for (int j = 0; j < 4; j++)
                if (r0 + tn + j < r_end) o[j] = accumulate ? o[j] + acc[i][j] : acc[i][j];
        }
    }
}

__device__ __forceinline__ float embed_to_f32(float v) { return v; }
__device__ __forceinline__ float embed_to_f32(__half v) { return __half2float(v); }
__device__ __forceinline__ float embed_to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

// Embedding gather: out[r][:] = table[rows[r]][:] widened to f32 (src/cpu_backend.cpp:33 does this with
// ops::dequant_row on the host). A row index outside the table gives zeros and raises *status.
template <typename W>
__global__ void embed_rows_kernel(float* out, const W* __restrict__ table, int n_in, int n_rows_table, const int32_t* __restrict__ rows,
                                  int* status, float scale) {
    const int row = rows[blockIdx.x];
    float* o = out + (size_t)blockIdx.x * n_in;
    if (row < 0 || row >= n_rows_table) {
        if (threadIdx.x == 0 && status) atomicOr(status, 1);
        for (int i = threadIdx.x; i < n_in; i += blockDim.x) o[i] = 0.f;
        return;
    }
    const W* src = table + (size_t)row * n_in;
    for (int i = threadIdx.x; i < n_in; i += blockDim.x) o[i] = embed_to_f32(src[i]) * scale;
}

// The same from two tables, added; `copy` (may be null) receives the rows too. A row index outside its table gives zeros and raises *status.
__global__ void embed_sum_kernel(float* out, float* copy, const __nv_bfloat16* __restrict__ table, int n_table, const int32_t* __restrict__ rows,
                                 const __nv_bfloat16* __restrict__ table2, int n_table2, const int32_t* __restrict__ rows2, int n, float scale, int* status) {
    const int a = rows[blockIdx.x], b = table2 ? rows2[blockIdx.x] : 0;
    const bool ok = a >= 0 && a < n_table && (!table2 || (b >= 0 && b < n_table2));
    if (!ok && threadIdx.x == 0) atomicOr(status, 1);
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        float v = ok ? __bfloat162float(table[(size_t)a * n + i]) : 0.f;
        if (ok && table2) v += __bfloat162float(table2[(size_t)b * n + i]);
        v *= scale;
        out[(size_t)blockIdx.x * n + i] = v;
        if (copy) copy[(size_t)blockIdx.x * n + i] = v;
    }
}

// [a | b] row by row, as f32 and / or as bf16 planes (lo may be null)
__global__ void concat_rows_kernel(float* f32, __nv_bfloat16* hi, __nv_bfloat16* lo, const float* a, const float* b, int n) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i >= 2 * n) return;
    const size_t row = blockIdx.y;
    const float4 v = i < n ? *reinterpret_cast<const float4*>(a + row * n + i) : *reinterpret_cast<const float4*>(b + row * n + i - n);
    const size_t at = row * 2 * n + i;
    if (f32) *reinterpret_cast<float4*>(f32 + at) = v;
    if (hi) {
        const __nv_bfloat162 h[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
        reinterpret_cast<__nv_bfloat162*>(hi + at)[0] = h[0];
        reinterpret_cast<__nv_bfloat162*>(hi + at)[1] = h[1];
        if (lo) {
            reinterpret_cast<__nv_bfloat162*>(lo + at)[0] = __floats2bfloat162_rn(v.x - __low2float(h[0]), v.y - __high2float(h[0]));
            reinterpret_cast<__nv_bfloat162*>(lo + at)[1] = __floats2bfloat162_rn(v.z - __low2float(h[1]), v.w - __high2float(h[1]));
        }
    }
}

// x = cap * tanh(x / cap)
__global__ void softcap_kernel(float* x, size_t n, float cap) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] = cap * tanhf(x[i] / cap);
}

}  // namespace

extern "C" {

cudaError_t ingot_support_embed_rows(float* out, const void* table, int is_f16, int n_in, int n_rows_table, const int32_t* rows_dev,
                                     int n_rows, int* status_dev, cudaStream_t s) {
    if (n_rows < 1 || n_in < 1) return cudaErrorInvalidValue;
    if (is_f16) embed_rows_kernel<__half><<<n_rows, 256, 0, s>>>(out, static_cast<const __half*>(table), n_in, n_rows_table, rows_dev, status_dev, 1.0f);
    else embed_rows_kernel<float><<<n_rows, 256, 0, s>>>(out, static_cast<const float*>(table), n_in, n_rows_table, rows_dev, status_dev, 1.0f);
    return cudaGetLastError();
}

cudaError_t ingot_support_rmsnorm(float* out, const float* x, const float* w, int n_rows, int n, float eps, cudaStream_t s) {
    rmsnorm_kernel<<<n_rows, 256, 0, s>>>(out, x, w, n, eps);
    return cudaGetLastError();
}

cudaError_t ingot_support_silu_mul(float* gate, const float* up, size_t n, cudaStream_t s) {
    silu_mul_kernel<<<unsigned((n + 255) / 256), 256, 0, s>>>(gate, up, n);
    return cudaGetLastError();
}

// One token: out_m (+)= W_m . x' for n_mat <= 3 matrices [n_out[m]][n_in] of one format that share x (see
// gemv_stream_kernel). fmt: 0 f16 rows, 1 Q8_0, 2 Q4_0 (ws[m] = the quant plane, scales[m] = the scale plane of a
// matrix repacked by ingot_quant_repack). norm_w != nullptr folds the RMS norm in; swiglu != 0 takes exactly two
// matrices of equal height (gate, up) and outs[0] receives silu(gate) * up. n_in must be a multiple of 256 (f16),
// 512 (Q8_0) or 1024 (Q4_0).
static cudaError_t gemv_group(float* const* outs, const void* const* ws, const void* const* scales, int fmt, const int* n_out, int n_mat,
                              int swiglu, int act, const float* x, const float* norm_w, float eps, int n_in, int n_mean, int accumulate,
                              cudaStream_t s) {
    const bool plain = fmt == kFmtF16 || fmt == kFmtBF16;
    const int chunk = plain ? 256 : fmt == kFmtQ8_0 ? 512 : 1024;
    if (fmt < 0 || fmt > 3 || n_mat < 1 || n_mat > 3 || n_in % chunk != 0 || n_in > kGemvMaxIn ||
        (swiglu && (n_mat != 2 || n_out[0] != n_out[1] || (!norm_w && fmt != kFmtBF16))) || (!plain && !scales))
        return cudaErrorInvalidValue;
    GemvGroup g = {};
    int total = 0;
    for (int m = 0; m < 3; m++) {
        const int mm = m < n_mat ? m : n_mat - 1;
        g.w[m] = ws[mm];
        g.d[m] = plain ? nullptr : static_cast<const __half*>(scales[mm]);
        g.out[m] = outs[mm];
        if (m < n_mat) total += n_out[m];
        g.row_end[m] = swiglu ? n_out[0] : total;
    }
    g.n_mat = n_mat;
    const int rows = swiglu ? n_out[0] : total;
    const size_t smem = (size_t)n_in * sizeof(float);
    // kLoads = 6 for short rows: with the current and the next step in flight the whole row is requested at once
    const bool short_rows = n_in / chunk <= 12;  // current and next step together cover the row
    typedef void (*Kernel)(GemvGroup, const float*, const float*, float, int, int, int, int, int, int);
    auto pick = [&](auto fmt_tag) -> Kernel {
        constexpr int F = decltype(fmt_tag)::value;
        if constexpr (F == kFmtBF16)
            if (swiglu && !norm_w) return short_rows ? gemv_stream_kernel<false, true, 6, F> : gemv_stream_kernel<false, true, 4, F>;
        return short_rows ? (swiglu ? gemv_stream_kernel<true, true, 6, F> : norm_w ? gemv_stream_kernel<true, false, 6, F> : gemv_stream_kernel<false, false, 6, F>)
                          : (swiglu ? gemv_stream_kernel<true, true, 4, F> : norm_w ? gemv_stream_kernel<true, false, 4, F> : gemv_stream_kernel<false, false, 4, F>);
    };
    Kernel kernel = fmt == kFmtBF16 ? pick(std::integral_constant<int, kFmtBF16>()) : fmt == kFmtF16 ? pick(std::integral_constant<int, kFmtF16>()) : fmt == kFmtQ8_0 ? pick(std::integral_constant<int, kFmtQ8_0>())
                                                                                               : pick(std::integral_constant<int, kFmtQ4_0>());
    // Environment knobs are process-wide and read once; the SM count belongs to the current device and is looked up
    // on every call (a cached attribute read), so that one process may drive several GPUs.
    static const bool use_pdl = getenv("INGOT_NO_PDL") == nullptr;
    // CTAs of one launch per SM. Fewer than fit leaves room for the next launch's CTAs, which then request
    // their first weights while this launch is still streaming (programmatic dependent launch).
    static const int ctas_per_sm_cap = [] { const char* c = getenv("INGOT_GEMV_CTAS_PER_SM"); return c ? atoi(c) : 0; }();
    int dev = 0, num_sms = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e == cudaSuccess) e = cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, dev);
    if (e != cudaSuccess) return e;
    int occ = 0;
    const int threads = plain ? StreamThreads<kFmtF16>::value : StreamThreads<kFmtQ8_0>::value, cta_warps = threads / 32;
    e = cudaOccupancyMaxActiveBlocksPerMultiprocessor(&occ, kernel, threads, smem);
    if (e != cudaSuccess) return e;
    if (occ < 1) occ = 1;
    if (ctas_per_sm_cap > 0) occ = occ < ctas_per_sm_cap ? occ : ctas_per_sm_cap;
    // One resident wave. Quantised rows: a CTA slot on every SM is used, the rows go round-robin over all warps (warps of
    // every CTA alike get the odd row more). f16 rows: as many warps as give every warp the same number of rows, which
    // leaves some SMs without a CTA but has no uneven tail - measured tg32 589 against 578 tok/s with the full grid,
    // while the quantised formats gain from it (Q8_0 561 -> 565, Q4_0 540 -> 554).
    int ctas;
    if (plain) {
        const int capacity = num_sms * occ * cta_warps;
        const int rows_per_warp = (rows + capacity - 1) / capacity;
        ctas = ((rows + rows_per_warp - 1) / rows_per_warp + cta_warps - 1) / cta_warps;
    } else {
        ctas = std::min(num_sms * occ, (rows + cta_warps - 1) / cta_warps);
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(ctas);
    cfg.blockDim = dim3(threads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = use_pdl ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, g, x, norm_w, eps, n_in, rows, accumulate, use_pdl ? 1 : 0, n_mean, act);
}

cudaError_t ingot_support_gemv_group(float* const* outs, const void* const* ws, const void* const* scales, int fmt, const int* n_out, int n_mat,
                                     int swiglu, const float* x, const float* norm_w, float eps, int n_in, int accumulate, cudaStream_t s) {
    if (fmt > 2) return cudaErrorInvalidValue;
    return gemv_group(outs, ws, scales, fmt, n_out, n_mat, swiglu, 0, x, norm_w, eps, n_in, n_in, accumulate, s);
}

// The same streaming kernel for one bf16 matrix [n_out][n_in] (n_in a multiple of 256): out (+)= W x', x' = rmsnorm(x) with the mean
// over n_mean floats if norm_w is given, else x itself. gated: W holds a gate and an up half of n_out rows each, out = act(gate) * up.
cudaError_t ingot_support_gemv_bf16(float* out, const void* w, int n_out, int n_in, const float* x, const float* norm_w, float eps, int n_mean,
                                    int gated, int act, int accumulate, cudaStream_t s) {
    float* outs[2] = {out, out};
    const void* ws[2] = {w, static_cast<const char*>(w) + (size_t)n_out * n_in * 2};
    const int rows[2] = {n_out, n_out};
    return gemv_group(outs, ws, nullptr, kFmtBF16, rows, gated ? 2 : 1, gated, act, x, norm_w, eps, n_in, n_mean, accumulate, s);
}

}  // extern "C"

namespace {
template <typename... KArgs, typename... Args>
cudaError_t support_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, Args&&... args) {
    static const bool use_pdl = getenv("INGOT_NO_PDL") == nullptr;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = use_pdl ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}

template <typename W>
cudaError_t launch_linear(float* out, const void* w, const float* x, int x_ld, int n_in, int n_out, int rows_per_block, int n_tok,
                          int accumulate, cudaStream_t s) {
    const int warps = 8;
    const W* wt = static_cast<const W*>(w);
    const XLayout xl = {x_ld, rows_per_block};
    if (std::is_same<W, __nv_bfloat16>::value && n_tok == 1 && rows_per_block == 0 && n_out <= 2048 && n_in >= 1024)
        return support_launch(gemv_row_kernel, dim3(n_out), dim3(256), 0, s, out, static_cast<const __nv_bfloat16*>(w), x, n_in, accumulate);
    if (n_tok == 1 && rows_per_block == 0) {
        const unsigned grid = (n_out + warps - 1) / warps;
        return support_launch(gemv_kernel<W>, dim3(grid), dim3(warps * 32), 0, s, out, wt, x, n_in, n_out, accumulate);
    }
    if (n_tok >= 16 && n_out % 4 == 0 && (rows_per_block == 0 || rows_per_block % 4 == 0)) {
        const int per = rows_per_block > 0 ? rows_per_block : n_out;
        dim3 grid((n_out / per) * ((per + kGN - 1) / kGN), (n_tok + kGM - 1) / kGM);
        return support_launch(gemm_kernel<W>, grid, dim3(256), 0, s, out, wt, x, n_in, n_out, n_tok, accumulate, xl);
    }
    if (n_tok == 1) {
        dim3 grid((n_out + warps - 1) / warps, 1);
        return support_launch(linear_kernel<W, 1>, grid, dim3(warps * 32), 0, s, out, wt, x, n_in, n_out, n_tok, accumulate, xl);
    }
    dim3 grid((n_out + warps - 1) / warps, (n_tok + 7) / 8);
    return support_launch(linear_kernel<W, 8>, grid, dim3(warps * 32), 0, s, out, wt, x, n_in, n_out, n_tok, accumulate, xl);
}
}  // namespace

extern "C" {

// w_is_f16: 1 = __half weights, 0 = float weights.
cudaError_t ingot_support_linear(float* out, const void* w, int w_is_f16, const float* x, int n_in, int n_out, int n_tok,
                                 int accumulate, cudaStream_t s) {
    return w_is_f16 ? launch_linear<__half>(out, w, x, n_in, n_in, n_out, 0, n_tok, accumulate, s)
                    : launch_linear<float>(out, w, x, n_in, n_in, n_out, 0, n_tok, accumulate, s);
}

// bf16 weights, f32 activations whose rows are x_ld floats apart (a multiple of 4, as is the offset of x), f32 products.
// rows_per_block > 0: block-diagonal (see XLayout). n_in a multiple of 8.
cudaError_t ingot_support_linear_bf16(float* out, const void* w, const float* x, int x_ld, int n_in, int n_out, int rows_per_block,
                                      int n_tok, int accumulate, cudaStream_t s) {
    if (n_in % 8 != 0 || x_ld % 4 != 0 || (rows_per_block > 0 && n_out % rows_per_block != 0)) return cudaErrorInvalidValue;
    return launch_linear<__nv_bfloat16>(out, w, x, x_ld, n_in, n_out, rows_per_block, n_tok, accumulate, s);
}

// Embedding rows of a bf16 table, widened to f32 and scaled (table rows n_in apart).
cudaError_t ingot_support_embed_rows_bf16(float* out, const void* table, int n_in, int n_rows_table, const int32_t* rows_dev, int n_rows,
                                          float scale, int* status_dev, cudaStream_t s) {
    if (n_rows < 1 || n_in < 1) return cudaErrorInvalidValue;
    embed_rows_kernel<__nv_bfloat16><<<n_rows, 256, 0, s>>>(out, static_cast<const __nv_bfloat16*>(table), n_in, n_rows_table, rows_dev, status_dev, scale);
    return cudaGetLastError();
}

// out[r][:] = rmsnorm(x[rows ? rows[r] : r]) over rows of n floats whose mean is taken over n_mean of them (rows padded with
// zeros up to n). rows may be null.
cudaError_t ingot_support_rmsnorm_rows(float* out, const float* x, const float* w, const int32_t* rows_dev, int n_rows, int n, int n_mean,
                                       float eps, cudaStream_t s) {
    return support_launch(rmsnorm_rows_kernel, dim3(n_rows), dim3(256), 0, s, out, x, w, rows_dev, n, n_mean, eps);
}

// out[r][i] = act(gate) * up with gate = in[r][i], up = in[r][n + i] (one product holds both halves); act: 0 silu, 1 gelu (tanh form)
cudaError_t ingot_support_gated_act(float* out, const float* in, int n_rows, int n, int act, cudaStream_t s) {
    const size_t total = (size_t)n_rows * n;
    return support_launch(gated_act_kernel, dim3(unsigned((total + 255) / 256)), dim3(256), 0, s, out, in, n, total, act);
}

// out[r] (and copy[r], may be null) = scale * (table[rows[r]] + table2[rows2[r]]) (table2 may be null); rows of n_in values.
cudaError_t ingot_support_embed_sum_bf16(float* out, float* copy, const void* table, int n_rows_table, const int32_t* rows_dev, const void* table2,
                                         int n_rows_table2, const int32_t* rows2_dev, int n_in, int n_rows, float scale, int* status_dev, cudaStream_t s) {
    if (n_rows < 1 || n_in < 1 || (table2 && !rows2_dev) || !status_dev) return cudaErrorInvalidValue;
    embed_sum_kernel<<<n_rows, 256, 0, s>>>(out, copy, static_cast<const __nv_bfloat16*>(table), n_rows_table, rows_dev,
                                            static_cast<const __nv_bfloat16*>(table2), n_rows_table2, rows2_dev, n_in, scale, status_dev);
    return cudaGetLastError();
}

// [a | b] of rows of n values (a multiple of 4) as f32 rows and / or bf16 planes; null pointers are skipped.
cudaError_t ingot_support_concat_rows(float* f32, void* hi, void* lo, const float* a, const float* b, int n, int n_rows, cudaStream_t s) {
    if (n < 4 || n % 4 != 0 || n_rows < 1) return cudaErrorInvalidValue;
    return support_launch(concat_rows_kernel, dim3(unsigned((2 * n / 4 + 255) / 256), n_rows), dim3(256), 0, s, f32, static_cast<__nv_bfloat16*>(hi),
                          static_cast<__nv_bfloat16*>(lo), a, b, n);
}

cudaError_t ingot_support_softcap(float* x, size_t n, float cap, cudaStream_t s) {
    return support_launch(softcap_kernel, dim3(unsigned((n + 255) / 256)), dim3(256), 0, s, x, n, cap);
}

}  // extern "C"
