// Residual sum with norms before and after it: the sum of a product's slices, of routed rows and of the part's own input, the norm of that
// result, the residual add, and the norm the next part reads x through, as f32 rows or as the bf16 operand of its products. One CTA per
// row, which stays in registers throughout; variances are means of squared deviations, taken in a second pass over the registers.
#include "residual_norm.h"

#include <cuda_bf16.h>

#include "../csrc/ingot_internal.cuh"

namespace {

__device__ __forceinline__ float block_sum(float v, float* red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    __syncthreads();  // red is free again
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    for (int w = 0; w < (int)(blockDim.x >> 5); w++) t += red[w];
    return t;
}

template <int kKeep>
struct Row {
    float4 v[kKeep];
};

// (mean, 1 / deviation) of the first n_mean values; the mean is 0 for norms that do not centre.
template <int kKeep>
__device__ __forceinline__ float2 moments(const Row<kKeep>& r, int n_mean, bool centred, float eps, float* red) {
    float mean = 0.f;
    if (centred) {  // the padding holds zeros
        float s = 0.f;
#pragma unroll
        for (int k = 0; k < kKeep; k++) s += (r.v[k].x + r.v[k].y) + (r.v[k].z + r.v[k].w);
        mean = block_sum(s, red) / float(n_mean);
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < kKeep; k++) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        const float d[4] = {r.v[k].x - mean, r.v[k].y - mean, r.v[k].z - mean, r.v[k].w - mean};
#pragma unroll
        for (int e = 0; e < 4; e++)
            if (i + e < n_mean) ss = fmaf(d[e], d[e], ss);
    }
    return make_float2(mean, 1.0f / sqrtf(block_sum(ss, red) / float(n_mean) + eps));
}
__device__ __forceinline__ float4 apply(float4 v, float2 m, const ingot_norm& n, int i) {
    const float4 w = *reinterpret_cast<const float4*>(n.w + i);
    float4 o = make_float4((v.x - m.x) * m.y * w.x, (v.y - m.x) * m.y * w.y, (v.z - m.x) * m.y * w.z, (v.w - m.x) * m.y * w.w);
    if (n.b) {
        const float4 b = *reinterpret_cast<const float4*>(n.b + i);
        o.x += b.x; o.y += b.y; o.z += b.z; o.w += b.w;
    }
    return o;
}

template <int kKeep, int kThreads>
__global__ void __launch_bounds__(kThreads) residual_norm_kernel(const ingot_residual_norm p) {
    __shared__ float red[32];
    INGOT_PDL_TRIGGER();
    INGOT_PDL_WAIT();
    const int row = blockIdx.x, step = blockDim.x * 4;
    float* xr = p.x + (size_t)(p.rows ? p.rows[row] : row) * p.n;
    Row<kKeep> x;
#pragma unroll
    for (int k = 0; k < kKeep; k++) {
        const int i = threadIdx.x * 4 + k * step;
        x.v[k] = i < p.n ? *reinterpret_cast<const float4*>(xr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (p.n_slices > 0 || p.top > 0 || p.self_gain) {
        Row<kKeep> y;
        const float gain = p.gain ? p.gain[row] : 1.0f;
        const size_t slice = (size_t)p.n_rows * p.n;
#pragma unroll
        for (int k = 0; k < kKeep; k++) {
            const int i = threadIdx.x * 4 + k * step;
            y.v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i >= p.n) continue;
            for (int s = 0; s < p.n_slices; s++) {
                const float4 a = *reinterpret_cast<const float4*>(p.product + s * slice + (size_t)row * p.n + i);
                y.v[k].x += a.x; y.v[k].y += a.y; y.v[k].z += a.z; y.v[k].w += a.w;
            }
            y.v[k].x *= gain; y.v[k].y *= gain; y.v[k].z *= gain; y.v[k].w *= gain;
        }
        for (int t = 0; t < p.top; t++) {
            const int r = p.row_of[(size_t)row * p.top + t];
            if (r < 0) continue;
#pragma unroll
            for (int k = 0; k < kKeep; k++) {
                const int i = threadIdx.x * 4 + k * step;
                if (i >= p.n) continue;
                const float4 a = *reinterpret_cast<const float4*>(p.branch + (size_t)r * p.n + i);
                y.v[k].x += a.x; y.v[k].y += a.y; y.v[k].z += a.z; y.v[k].w += a.w;
            }
        }
        const float self = p.self_gain ? p.self_gain[row] : 0.f;
        if (self != 0.f) {  // block-uniform
            const float2 m = moments(x, p.n_mean, p.self.b != nullptr, p.eps, red);
#pragma unroll
            for (int k = 0; k < kKeep; k++) {
                const int i = threadIdx.x * 4 + k * step;
                if (i >= p.n) continue;
                const float4 h = apply(x.v[k], m, p.self, i);
                y.v[k].x = fmaf(self, h.x, y.v[k].x); y.v[k].y = fmaf(self, h.y, y.v[k].y);
                y.v[k].z = fmaf(self, h.z, y.v[k].z); y.v[k].w = fmaf(self, h.w, y.v[k].w);
            }
        }
        if (p.post.w) {
            const float2 m = moments(y, p.n_mean, p.post.b != nullptr, p.eps, red);
#pragma unroll
            for (int k = 0; k < kKeep; k++) {
                const int i = threadIdx.x * 4 + k * step;
                if (i < p.n) y.v[k] = apply(y.v[k], m, p.post, i);
            }
        }
#pragma unroll
        for (int k = 0; k < kKeep; k++) {
            const int i = threadIdx.x * 4 + k * step;
            x.v[k].x += y.v[k].x; x.v[k].y += y.v[k].y; x.v[k].z += y.v[k].z; x.v[k].w += y.v[k].w;
            if (i < p.n) *reinterpret_cast<float4*>(xr + i) = x.v[k];
        }
    }
    if (!p.next.w) return;
    const float2 m = moments(x, p.n_mean, p.next.b != nullptr, p.eps, red);
#pragma unroll
    for (int k = 0; k < kKeep; k++) {
        const int i = threadIdx.x * 4 + k * step;
        if (i >= p.n) continue;
        const float4 v = apply(x.v[k], m, p.next, i);
        const size_t at = (size_t)row * p.n + i;
        if (p.out) *reinterpret_cast<float4*>(p.out + at) = v;
        if (p.hi) {
            const __nv_bfloat162 h[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
            *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p.hi) + at) = *reinterpret_cast<const uint2*>(h);
            if (p.lo) {
                const __nv_bfloat162 l[2] = {__floats2bfloat162_rn(v.x - __low2float(h[0]), v.y - __high2float(h[0])),
                                             __floats2bfloat162_rn(v.z - __low2float(h[1]), v.w - __high2float(h[1]))};
                *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p.lo) + at) = *reinterpret_cast<const uint2*>(l);
            }
        }
    }
}

}  // namespace

extern "C" cudaError_t ingot_residual_norm_run(const ingot_residual_norm* r, cudaStream_t s) {
    if (!r->x || r->n < 4 || r->n % 4 != 0 || r->n_mean < 1 || r->n_mean > r->n || r->n_rows < 1 || (r->n_slices > 0 && !r->product) ||
        (r->top > 0 && (!r->branch || !r->row_of)) || (r->self_gain && !r->self.w) || (r->next.w && !r->out && !r->hi))
        return cudaErrorInvalidValue;
    auto run = [&](auto kernel, int threads) { return ingot_launch_pdl(kernel, dim3(r->n_rows), dim3(threads), 0, s, *r); };
    const int quads = r->n / 4;
    auto warps = [&](int keep) { return (quads + 32 * keep - 1) / (32 * keep) * 32; };  // threads that hold a row of `keep` quads each
    if (quads <= 256) return run(residual_norm_kernel<1, 256>, warps(1));
    if (quads <= 1024) return run(residual_norm_kernel<4, 256>, warps(4));
    if (quads <= 2048) return run(residual_norm_kernel<8, 256>, 256);
    if (quads <= 8192) return run(residual_norm_kernel<8, 1024>, 1024);
    return cudaErrorInvalidValue;
}
