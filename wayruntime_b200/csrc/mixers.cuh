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

// x[r] = scale * table[token[r]] (+ sinusoidal position vector; turns[i] = frequency of pair i in turns per token)
int wr_embed_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const uint32_t *tokens, const void *table, int table_type,
                    const double *turns, float *x, uint32_t width, float scale);

struct wr_norm_args {
    const float *x;                  // [rows][wr_ld(width)]
    const uint32_t *gather;          // row r reads x row gather[r], or null
    const float *w, *shift;          // norm weight; token-shift weight or null
    uint64_t state_off;              // where the previous token's row is kept in the state (with shift)
    uint32_t width, groups;
    float eps;
    bool centre;                     // layer norm: the group's mean comes off first
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
    bool shared;                         // a key's first vd numbers are its value (v_dim 0 in the cache)
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

// ---- mixture of experts (moe.cu): routing

// The chosen experts of every row and their weights, and the rows grouped by expert.  Many rows: expert e's (row, slot)
// pairs take consecutive places from a multiple of `tile` on; list names the expert of each tile of places.  Few
// rows: list names the experts somebody chose, and a pair's place is its expert's number in the list.
struct wr_route_args {
    const float *logits;             // [rows][ld]
    uint32_t ld;
    const float *bias;               // [experts]
    uint32_t experts, top, tile;     // tile 0: few rows
    float *weight;                   // [rows][top]
    uint32_t *expert, *place;        // [rows][top]
    uint32_t *row_of;                // [places]: the row at a place, ~0 where there is none (many rows)
    uint32_t *list, *count;
    bool chosen;                     // another kernel has done so already (many rows: their places are still to be found)
};
inline uint32_t wr_route_tiles(uint32_t rows, uint32_t experts, uint32_t top, uint32_t tile)
{
    const uint32_t pairs = rows * top, used = experts < pairs ? experts : pairs;
    return tile ? pairs / tile + used : used;
}
// ---- attention over a latent (latent.cu)

// Where the parts of a latent layer's rows lie: the cached row is [latent, padded to 64 | rotated key part, padded to
// 64], a head's query [unrotated, padded to 16 | rotated, padded to 16].
struct wr_latent_geom {
    uint32_t heads, dim, rot, vdim, q_rank, kv_rank;
    __host__ __device__ uint32_t dim_pad() const { return (dim + 15u) & ~15u; }
    __host__ __device__ uint32_t rot_pad() const { return (rot + 15u) & ~15u; }
    __host__ __device__ uint32_t vdim_pad() const { return (vdim + 15u) & ~15u; }
    __host__ __device__ uint32_t q_head() const { return dim_pad() + rot_pad(); }
    __host__ __device__ uint32_t rank_pad() const { return (kv_rank + 63u) & ~63u; }
    __host__ __device__ uint32_t row() const { return rank_pad() + ((rot + 63u) & ~63u); }
};

// Heads that share a cached row's fetch in attn_latent.cu, and the queries as its operand: per row and group of heads, boxes
// of 64 columns, each [2 group][128 B] in the 128-byte swizzle — the heads' F16 roundings, then what is left of them.
__host__ __device__ inline uint32_t wr_latent_group(const wr_latent_geom &g) { return g.heads <= 8 ? 8u : 16u; }
__host__ __device__ inline size_t wr_latent_split_bytes(const wr_latent_geom &g)
{
    const uint32_t nh = wr_latent_group(g);
    return (size_t)((g.heads + nh - 1) / nh) * (2 * nh) * g.row() * 2;
}
__host__ __device__ inline uint32_t wr_latent_split_off(uint32_t rows, uint32_t r, uint32_t c)
{
    return (c >> 6) * rows * 128u + r * 128u + ((((c & 63u) >> 3) ^ (r & 7u)) << 4) + (c & 7u) * 2u;
}

// The projection's rows, normed and rotated: the query latent for the next product, and (own) the session's row.
struct wr_latent_prep_args {
    wr_latent_geom g;
    const float *in;                 // [rows][ld]: query latent at 0, latent at c_off, rotated key part at r_off
    uint32_t ld, c_off, r_off;
    const float *q_norm, *c_norm;
    float eps;
    const double *turns;             // [rot/2] frequencies in turns per token
    void *cq; int cq_type;           // [rows][wr_ld(q_rank)]
    bool own;
    uint32_t layer;                  // page-table layer
    wr_kv_geom kv;
    const wr_route_args *route;      // the rows' experts chosen on the way, or null
};
int wr_latent_prep_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_prep_args &a);

// Queries moved into the latent: out[row][head] = scale [w_uk^T q | rotated q], padded as the cached row.  w_ukv:
// dim_pad() key rows per head, then vdim_pad() value rows per head; F32 rows wr_ld(kv_rank) apart or F16 in blocks
// (wr_weight).
struct wr_latent_query_args {
    wr_latent_geom g;
    const float *q;                  // [rows][heads][q_head()]
    const void *w_ukv; int w_type;   // WR_ACT_F32 / WR_ACT_F16
    const double *turns;
    float scale;
    bool split;                      // at most WR_CUDA_BATCH_MAX rows, F16 weights: out is the split operand above, in log2 units
    float *out;                      // [rows][heads][row()]
};
int wr_latent_query_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_query_args &a);

// Latent attention rows back into values: out[row][head * vdim + v] = w_uv o.
struct wr_latent_lens {
    uint32_t len[WR_CUDA_BATCH_MAX], count[WR_CUDA_BATCH_MAX];   // keys a row sees; chunks they were cut into
};
struct wr_latent_value_args {
    wr_latent_geom g;
    const float *o;                  // [rows][heads][kv_rank]; split: rank_pad() values each
    bool split;                      // at most WR_CUDA_BATCH_MAX rows, F16 weights, split rows out
    const float *ml;                 // split: o is still in chunks, [rows][heads][chunks][rank_pad()], with these pairs; or null
    uint32_t chunks;
    wr_latent_lens lens;
    const void *w_ukv; int w_type;
    void *out; int out_type;         // [rows][out_ld]; the columns up to wr_ld(heads * vdim) are written
    uint32_t out_ld;
};
int wr_latent_value_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_value_args &a);

// Causal attention of a prompt's rows on the tensor cores (attn_prefill.cu), with keys and values written out per head.
struct wr_latent_flash_args {
    wr_latent_geom g;
    uint32_t n, p0;                  // rows, and where they start in the session
    const void *q;                   // F16 [n][heads][q_head()], rotated
    const void *kv;                  // F16 [p0 + n][heads * dim_pad() keys, then heads * vdim_pad() values]
    const uint64_t *pages;           // device page table of the rows (their rotated key part)
    float scale;
    void *out;                       // BF16 [n][out_ld]; the columns up to wr_ld(heads * vdim) are written
    uint32_t out_ld;
};
bool wr_latent_flash_covers(const wr_latent_geom &g, float scale);
int wr_latent_flash_launch(wr_cuda_ctx *ctx, const wr_latent_flash_args &a);

// Attention of at most WR_CUDA_BATCH_MAX rows over the cached F16 rows (attn_latent.cu): q as wr_latent_query_launch leaves
// it with `split`, lens: how many keys each row sees (host).  Fills in out's o, ml, chunks and lens; merged: room for
// [rows][heads][rank_pad()].
bool wr_latent_decode_covers(const wr_latent_geom &g);
int wr_latent_decode_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_geom &g, uint32_t layer, const void *q,
                            const uint32_t *lens, float *merged, wr_latent_value_args &out);

// q's rotated parts turned in place (F16 rows as above)
int wr_latent_rotate_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_geom &g, const double *turns, void *q);

// ---- mixture of experts (moe.cu)

int wr_route_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_route_args &a);

// out[place] = x[row_of[place]] (BF16 rows of ld values)
int wr_moe_gather_launch(wr_cuda_ctx *ctx, const void *x, void *out, uint32_t ld, const uint32_t *row_of,
                         const uint32_t *count, uint32_t max_tiles, uint32_t tile);

// resid[row] += mul * sum over slots of weight * y[place], slots in order
struct wr_combine_args {
    const void *y; int type;         // [places][ld]; few rows: F32, place's row r at 16 place + r
    uint32_t ld, width, top;
    bool few;
    const float *weight;
    const uint32_t *place;
    float mul;
    float *resid;                    // [rows][ld]
};
int wr_moe_combine_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_combine_args &a);

// F32 experts: out[place] = act(gate x, up x) (up != null) or gate x, tiles of kMoeTileF32 places; x rows through row_of
// or (null) places themselves.
constexpr uint32_t kMoeTileF32 = 32;
struct wr_moe_f32_args {
    const float *x, *gate, *up;      // weights of expert 0; those of expert e at e * stride floats
    size_t stride;
    uint32_t x_ld, n, k, out_ld;     // rows of weights wr_ld(k) apart
    float alpha, limit;
    const uint32_t *row_of, *list, *count;
    uint32_t max_tiles;
    float *out;
};
int wr_moe_f32_launch(wr_cuda_ctx *ctx, const wr_moe_f32_args &a);
