// gemv.cuh — the weight-streaming matrix product for a few activation rows, shared by the model stacks.
#pragma once

#include "wr_internal.cuh"

struct GemvSeg {
    const float *w;        // [n][k] row-major (GGML layout of a [k -> n] weight)
    float *out;            // [rows][out_stride]
    uint32_t n, out_stride;
};

enum { WR_GEMV_ACT_NONE = 0, WR_GEMV_ACT_SOFTPLUS = 1 };

struct GemvParams {
    GemvSeg seg[3];
    uint32_t cta_end[3];   // running CTA count after each segment (filled by wr_gemv_launch)
    uint32_t n_seg;
    const float *x;        // [rows][x_stride]
    uint32_t x_stride, k, rows;
    const float *norm_w;   // fused RMSNorm weight over k, or null
    float eps;
    const float *add;      // residual rows added to the result, or null (may alias out)
    uint32_t add_stride;
    uint32_t swiglu;       // seg[0] = gate, seg[1] = up: seg[0].out <- SiLU(gate) * up
    const float *bias;     // added to segment 0's result, or null
    uint32_t act;          // WR_GEMV_ACT_* on the result (after the bias)
    float mul = 1.f;       // on the result before the residual
};

// Enqueue y[r][n] = sum_k W[n][k] x[r][k] on the context's stream (k a multiple of 4).  `width` is the output width
// the tiling is chosen by.
int wr_gemv_launch(wr_cuda_ctx *ctx, GemvParams &p, uint32_t width);
