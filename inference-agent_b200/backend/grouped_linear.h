// Grouped bf16 product (linear_sm100.cu): one weight matrix per run of rows.
#pragma once

#include <cuda_runtime.h>
#include <stdint.h>

struct ingot_linear_ws;

struct ingot_grouped_gemm {
    const void *a_hi, *a_lo;       // bf16 activation rows [n_rows][n_in], sorted by group; a_lo null: one plane
    int n_rows, rows_per_group;    // rows_per_group: the most rows a group can have
    const void* w;                 // bf16 [n_groups][n_out][n_in]
    int n_in, n_out, n_groups;     // lengths are multiples of 8
    const int32_t* group_start;    // device, [n_groups + 1]
    const float* row_scale;        // device, [n_rows]: multiplies the accumulator (null: none), then
    int act;                       // INGOT_ACT_*; SILU_GATED: n_out counts gate and up columns (runs of 32 of each), the result is half as wide
                                   // and the factor follows the activation
    float* out;                    // f32 [n_rows][n_out], or
    void *out_hi, *out_lo;         // bf16 plane(s) of the same shape (out_hi non-null)
};

extern "C" cudaError_t ingot_grouped_tc_run(ingot_linear_ws* ws, const ingot_grouped_gemm* g, cudaStream_t s);
