// gemm_bf16.cuh — BF16 tensor-core matrix product for many activation rows (prefill of the mixed stack).
#pragma once

#include <cuda.h>

#include "wr_internal.cuh"

enum { WR_GEMM_OUT_F32 = 0, WR_GEMM_OUT_BF16 = 1, WR_GEMM_OUT_F16 = 2 };
enum { WR_GEMM_ACT_NONE = 0, WR_GEMM_ACT_SOFTPLUS = 1 };

// Gate and up products of a gated feed-forward in one: weight rows from `from` on come in groups of sixteen, eight
// gate rows and then the eight up rows that belong to them, and what leaves is act(gate, up), eight values a group.
enum { WR_PAIR_SILU = 0, WR_PAIR_LIMITED = 1 };
struct wr_pair_args {
    uint32_t from = ~0u;   // a multiple of 16; ~0: there are none
    uint32_t act = WR_PAIR_SILU;
    float alpha = 1.f, limit = 0.f;      // WR_PAIR_LIMITED: g sigmoid(alpha g) (u + 1), g <= limit, |u| <= limit
    void *out = nullptr;   // rows of BF16 values (many rows), or split rows (few)
    uint32_t ld = 0;
};
// One product per group of rows, each with a weight of its own (experts), `stride` bytes apart.  `list` names the
// weight of every 128-row tile of the activations (many rows), or of every group (few rows: group g's results are
// rows 16 g .. of out, split rows 32 g .. of pair.out, and its input the split rows x_rows * g ..).
struct wr_group_args {
    const uint32_t *list = nullptr;      // device memory, as is:
    const uint32_t *count = nullptr;     // how many entries the list has
    uint32_t max = 0;                    // at most this many
    uint32_t usual = 1;                  // few rows: how many a single row has
    uint32_t x_rows = 0;
    size_t stride = 0;
};

struct wr_gemm_args {
    uint32_t m;
    void *out;             // [m][out_ld] of out_type; out_ld a multiple of 8, at least w.n
    uint32_t out_ld, out_type;
    void *out_bf16;        // a second copy of the result in BF16 (before the residual), or null
    uint32_t out_bf16_ld;
    const float *bias;     // [w.n rounded up to 8] or null
    uint32_t act;          // WR_GEMM_ACT_* after the bias
    const float *add;      // [m][add_ld] residual added last (may alias an F32 out), or null
    uint32_t add_ld;
    float mul = 1.f;       // on the result before the residual
    wr_pair_args pair;
    wr_group_args group;   // m: rows the buffers hold
    // Activations out of a cache instead: row r is row r % 64 of page r / 64 (F16 blocks of 64 rows x 64 values, one after
    // the other from the page's start on), and the weight holds F16 values.
    const uint64_t *pages = nullptr;
};

// A BF16 weight [n][k] as the tensor core reads it: blocks of 64 rows x 64 K-values, each the 8 KB image of a
// 128-byte-swizzled operand (row r at r * 128, its 16-byte piece c at c ^ (r & 7)), K-blocks of a row block one
// after the other.  A block is one linear bulk copy, and a CTA's walk along K is one contiguous read.  Rows and
// K-values beyond n and k are zeros.
constexpr uint32_t kWBlock = 64, kWBlockBytes = kWBlock * kWBlock * 2;
struct wr_weight {
    const void *blocks;
    uint32_t n, k;
};
__host__ __device__ inline uint32_t wr_weight_blocks(uint32_t n) { return (n + kWBlock - 1) / kWBlock; }
inline size_t wr_weight_bytes(uint32_t n, uint32_t k) { return (size_t)wr_weight_blocks(n) * wr_weight_blocks(k) * kWBlockBytes; }
// byte offset of element (r, i)
__host__ __device__ inline size_t wr_weight_off(uint32_t k, uint32_t r, uint32_t i)
{
    const size_t block = (size_t)(r / kWBlock) * wr_weight_blocks(k) + i / kWBlock;
    const uint32_t rr = r % kWBlock, ii = i % kWBlock;
    return block * kWBlockBytes + rr * 128u + (((ii >> 3) ^ (rr & 7u)) << 4) + (ii & 7u) * 2u;
}

// Tensor map of activation rows [rows][k], ld elements apart (a multiple of 8; base 16-byte aligned).
// WR_CUDA_ERR_INTERNAL when the driver refuses the map.
int wr_gemm_map_rows(CUtensorMap *map, const void *x, uint32_t rows, uint32_t k, uint32_t ld);

// Enqueue out[m][n] = act(x . w^T + bias) + add on the context's stream.
int wr_gemm_launch(wr_cuda_ctx *ctx, const CUtensorMap &x, const wr_weight &w, const wr_gemm_args &args);

// The same product for at most WR_CUDA_BATCH_MAX rows, weights streamed once.  The activation rows are "split": an
// F32 value is kept as two BF16 numbers, its rounding in row r and what is left in row WR_CUDA_BATCH_MAX + r of one
// buffer, so the product sees about 16 bits of it.  A row's bits do not depend on the other rows.  out F32.
struct wr_skinny_args {
    uint32_t rows;
    float *out;            // [rows][out_ld]
    uint32_t out_ld;
    void *out_split;       // the result (before the residual) as split rows too, or null
    uint32_t out_split_ld;
    const float *bias;     // [n] or null
    uint32_t act;          // WR_GEMM_ACT_*
    const float *add;      // [rows][add_ld] or null (may alias out)
    uint32_t add_ld;
    float mul = 1.f;       // on the result before the residual
    wr_pair_args pair;
    wr_group_args group;
};
int wr_skinny_map_rows(CUtensorMap *map, const void *split_rows, uint32_t k, uint32_t ld, uint32_t groups = 1);
int wr_skinny_launch(wr_cuda_ctx *ctx, const CUtensorMap &x, const wr_weight &w, const wr_skinny_args &args);

#ifdef __CUDACC__
// act(gate, up) of wr_pair_args (the exponential and the quotient are the short sequences)
__device__ __forceinline__ float wr_pair_act(uint32_t act, float alpha, float limit, float g, float u)
{
    if (act == WR_PAIR_SILU) return __fdividef(g, 1.0f + __expf(-g)) * u;
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return __fdividef(g, 1.0f + __expf(-alpha * g)) * (u + 1.0f);
}
#endif
