// gemm_bf16.cuh — BF16 tensor-core matrix product for many activation rows (prefill of the mixed stack).
#pragma once

#include <cuda.h>

#include "wr_internal.cuh"

enum { WR_GEMM_OUT_F32 = 0, WR_GEMM_OUT_BF16 = 1, WR_GEMM_OUT_F16 = 2 };
enum { WR_GEMM_ACT_NONE = 0, WR_GEMM_ACT_SOFTPLUS = 1 };

struct wr_gemm_args {
    uint32_t m, n, k;
    void *out;             // [m][out_ld] of out_type; out_ld a multiple of 8, at least n
    uint32_t out_ld, out_type;
    void *out_bf16;        // a second copy of the result in BF16 (before the residual), or null
    uint32_t out_bf16_ld;
    const float *bias;     // [n rounded up to 8] or null
    uint32_t act;          // WR_GEMM_ACT_* after the bias
    const float *add;      // [m][add_ld] residual added last (may alias an F32 out), or null
    uint32_t add_ld;
};

// Tensor maps of the operands: a weight [n][k] with rows ld elements apart, and activation rows [rows][k].
// ld a multiple of 8, base 16-byte aligned.  WR_CUDA_ERR_INTERNAL when the driver refuses the map.
int wr_gemm_map_weight(CUtensorMap *map, const void *w, uint32_t n, uint32_t k, uint32_t ld);
int wr_gemm_map_rows(CUtensorMap *map, const void *x, uint32_t rows, uint32_t k, uint32_t ld);

// Enqueue out[m][n] = act(x . w^T + bias) + add on the context's stream.
int wr_gemm_launch(wr_cuda_ctx *ctx, const CUtensorMap &x, const CUtensorMap &w, const wr_gemm_args &args);

// The same product for at most WR_CUDA_BATCH_MAX rows, weights streamed once.  The activation rows are "split": an
// F32 value is kept as two BF16 numbers, its rounding in row r and what is left in row WR_CUDA_BATCH_MAX + r of one
// buffer, so the product sees about 16 bits of it.  A row's bits do not depend on the other rows.  out F32.
struct wr_skinny_args {
    uint32_t rows, n, k;
    float *out;            // [rows][out_ld]
    uint32_t out_ld;
    void *out_split;       // the result (before the residual) as split rows too, or null
    uint32_t out_split_ld;
    const float *bias;     // [n] or null
    uint32_t act;          // WR_GEMM_ACT_*
    const float *add;      // [rows][add_ld] or null (may alias out)
    uint32_t add_ld;
};
int wr_skinny_map_rows(CUtensorMap *map, const void *split_rows, uint32_t k, uint32_t ld);
int wr_skinny_launch(wr_cuda_ctx *ctx, const CUtensorMap &x, const CUtensorMap &w, const wr_skinny_args &args);
