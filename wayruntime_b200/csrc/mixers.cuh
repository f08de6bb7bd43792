// mixers.cuh — row kernels of the mixed layer stack: embedding, norms, token shift, convolution, selective
// scan, attention around the framework's cache.  Each is one mechanism with its constants as parameters.
#pragma once

#include "wr_internal.cuh"

// One session of a step, as the kernels see it.  In a decode step row r is the one token of session r; in a
// prefill step every row belongs to session 0.
struct wr_seq_dev {
    const uint64_t *pages;           // the session's page table, [layer][page]
    const char *st_in;               // recurrent state the step starts from
    char *st_out;                    // ... and where it leaves the new one
    uint32_t pos, n;                 // first position, tokens of this step
    uint32_t fresh;                  // no state yet: zeros
    uint32_t n_pages;                // pages per layer in the table
};
struct wr_rows {
    const wr_seq_dev *seqs;
    uint32_t n_rows, n_seq, decode;
};

// element types of activation rows
enum { WR_ACT_F32 = 0, WR_ACT_BF16 = 1, WR_ACT_F16 = 2, WR_ACT_SPLIT = 3 };    // SPLIT: see gemm_bf16.cuh

__host__ __device__ inline uint32_t wr_ld(uint32_t n) { return (n + 7u) & ~7u; }   // row stride of n values

// x[r] = table[token[r]] (+ sinusoidal position vector; turns[i] = frequency of pair i in turns per token)
int wr_embed_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const uint32_t *tokens, const void *table, int table_type,
                    const double *turns, float *x, uint32_t width);

struct wr_norm_args {
    const float *x;                  // [rows][wr_ld(width)]
    const uint32_t *gather;          // row r reads x row gather[r], or null
    const float *w, *shift;          // norm weight; token-shift weight or null
    uint64_t state_off;              // where the previous token's row is kept in the state (with shift)
    uint32_t width, groups;
    float eps;
    void *out;                       // [rows][wr_ld(width)] of out_type
    int out_type;
};
int wr_group_norm_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_norm_args &a);

struct wr_polynorm_args {
    const void *z; int z_type;       // [rows][wr_ld(ff)]
    void *out; int out_type;
    uint32_t ff;
    float a, b, c, e, eps;
};
int wr_polynorm_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_polynorm_args &a);

struct wr_conv_args {
    const void *x; int type;         // [rows][x_ld], channels first
    uint32_t x_ld, inner, taps;
    const float *w, *b;              // [taps][wr_ld(inner)] (tap-major), [inner]
    uint64_t state_off;              // [taps-1][wr_ld(inner)] F32
    void *out;                       // [rows][wr_ld(inner)] of `type`
    void *out_split;                 // the same as split rows too, or null (F32 only)
};
int wr_conv_silu_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_conv_args &a);

struct wr_scan_args {
    const void *x, *z; int type;     // [rows][x_ld], [rows][z_ld]
    uint32_t x_ld, z_ld;
    const float *dt;                 // [rows][wr_ld(inner)]
    const float *bc;                 // row r: B at b_off, C at c_off (multiples of 4), stride bc_ld
    uint32_t bc_ld, b_off, c_off;
    const float *a2;                 // [inner][wr_ld(state)]: -exp(A_log) log2(e), zero beyond state
    const float *d;                  // [inner]
    uint32_t inner, state;
    uint64_t state_off;              // [inner][state] F32
    void *out; int out_type;         // [rows][wr_ld(inner)]
};
int wr_scan_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_scan_args &a);

struct wr_attn_geom {
    uint32_t n_q, n_kv, maps, kd, vd;    // query heads, kv heads, maps per head, query/key size per map, value size
    uint32_t layer;                      // page-table layer
    wr_kv_geom kv;                       // the cache's layout (k_dim >= maps*kd, v_dim >= vd)
    bool hd128;                          // served by the head_dim-128 kernels: queries zero-padded to 128
    __host__ __device__ uint32_t vq() const { return n_q * maps; }               // queries per row
    __host__ __device__ uint32_t q_stride() const { return hd128 ? 128u : kd; }
    __host__ __device__ uint32_t o_stride() const { return hd128 ? 128u : vd; }
};
struct wr_attn_prep_args {
    wr_attn_geom g;
    const void *qkv; int type;       // [rows][ld]: q at 0, k at k_off, v at v_off
    uint32_t ld, k_off, v_off;
    float scale, temp_coef;          // q is multiplied by scale and, temp_every > 0, by its temperature
    uint32_t temp_every;
    void *q; int q_type;             // [rows][vq][q_stride]
};
int wr_attn_prep_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_attn_prep_args &a);

// Attention over the cache for layouts other than F16 head_dim 128.  q F32 [rows][vq][kd] with the scale folded
// in; out F32 [rows][vq][vd], normalised.  max_len: the longest session's length after this step.
int wr_attn_any_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_attn_geom &g, const float *q, float *out,
                       uint32_t max_len);

struct wr_attn_finish_args {
    wr_attn_geom g;
    const float *o;                  // [rows][vq][o_stride]
    float lambda, diff_init, eps;    // maps = 2
    const void *gate; int gate_type; // [rows][gate_ld], or null
    uint32_t gate_ld;
    void *out; int out_type;         // [rows][wr_ld(n_q*vd)]
};
int wr_attn_finish_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_attn_finish_args &a);
