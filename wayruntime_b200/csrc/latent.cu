// latent.cu — what surrounds attention over a shared latent row: norms and rotation of the projection, queries moved
// into the latent's space, and the attended latent turned back into values.
//
// All arithmetic is F32 (angles reduced in double).  A row's result depends on its session alone; the sums of an
// output follow one order whatever the number of rows.
#include <algorithm>

#include "gemm_bf16.cuh"
#include "latent_dev.cuh"
#include "moe_dev.cuh"
#include "rows_dev.cuh"
#include "warp_reduce.cuh"

namespace {

constexpr uint32_t kPrepThreads = 256, kTileRows = 16;           // (prompts: half as many)

__device__ __forceinline__ void angle(double turns, uint32_t pos, float &sn, float &cs)
{
    const double a = turns * (double)pos;                // in turns, reduced before it leaves double
    sincospif(2.0f * (float)(a - rint(a)), &sn, &cs);
}

// grid.y 0: the query latent; 1 (own): the session's row; the last (routed): the row's experts, of few rows all at once
template <typename TO>
__global__ void __launch_bounds__(kPrepThreads) latent_prep_kernel(const wr_rows rw, const wr_latent_prep_args a, const wr_route_args route)
{
    extern __shared__ float sm_prep[];
    __shared__ float part[kPrepThreads / 32];
    pdl_trigger();
    pdl_wait();
    const uint32_t row = blockIdx.x, n = blockIdx.y ? a.g.kv_rank : a.g.q_rank;
    if (blockIdx.y == (a.own ? 2u : 1u)) {
        if (route.tile == 0) {
            if (row == 0) route_few(sm_prep, route, rw.n_rows);
        } else if (threadIdx.x < 32) {
            choose(sm_prep, route, row);
        }
        return;
    }
    const float *in = a.in + (size_t)row * a.ld, *x = in + (blockIdx.y ? a.c_off : 0u);
    const float *w = blockIdx.y ? a.c_norm : a.q_norm;
    // pieces of eight; the pad columns of the projection and of the weights are zeros
    float ss = 0.f, v[8], u[8];
    for (uint32_t i = 8 * threadIdx.x; i < n; i += 8 * blockDim.x) {
        load8v(x + i, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, part) / (float)n + a.eps);
    auto scaled = [&](uint32_t i) {
        load8v(x + i, v);
        load8v(w + i, u);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= inv * u[e];
    };
    if (blockIdx.y == 0) {
        const Out<TO> out(a.cq, row, wr_ld(n));
        for (uint32_t i = 8 * threadIdx.x; i < n; i += 8 * blockDim.x) {
            scaled(i);
            out.put8(i, v);
        }
        return;
    }
    const wr_seq_dev s = rw.seqs[seq_of(rw, row)];
    const uint32_t pos = s.pos + tok_of(rw, row), tok = pos % kPageTokens, half = a.g.rot / 2;
    char *page = reinterpret_cast<char *>(s.pages[(size_t)a.layer * s.n_pages + pos / kPageTokens]);
    for (uint32_t i = 8 * threadIdx.x; i < n; i += 8 * blockDim.x) {
        scaled(i);
        char *p = page + wr_geom_off(a.kv, 0, 0, tok, i);
        if (a.kv.elem == WR_CUDA_F32) store8v(reinterpret_cast<float *>(p), v);
        else store8v(reinterpret_cast<__half *>(p), v);
    }
    auto put = [&](uint32_t d, float y) {
        char *p = page + wr_geom_off(a.kv, 0, 0, tok, d);
        if (a.kv.elem == WR_CUDA_F32) *reinterpret_cast<float *>(p) = y;
        else *reinterpret_cast<__half *>(p) = from_f32<__half>(y);
    };
    const float *r = in + a.r_off;
    for (uint32_t i = blockDim.x - 1 - threadIdx.x; i < half; i += blockDim.x) {         // (by threads without a piece first)
        float sn, cs;
        angle(a.turns[i], pos, sn, cs);
        put(a.g.rank_pad() + i, r[i] * cs - r[i + half] * sn);
        put(a.g.rank_pad() + half + i, r[i + half] * cs + r[i] * sn);
    }
}

// One block per row: the row's angles once, then every head's pairs.
__global__ void __launch_bounds__(256) latent_rotate_kernel(const wr_rows rw, const wr_latent_geom g, const double *turns, __half *q)
{
    __shared__ float2 turn[128];
    pdl_trigger();
    pdl_wait();
    const uint32_t row = blockIdx.x, half = g.rot / 2, hs = g.q_head();
    const uint32_t pos = rw.seqs[seq_of(rw, row)].pos + tok_of(rw, row);
    for (uint32_t i = threadIdx.x; i < half; i += 256) angle(turns[i], pos, turn[i].y, turn[i].x);
    __syncthreads();
    __half *base = q + (size_t)row * g.heads * hs + g.dim_pad();
    if (half % 2 == 0) {
        for (uint32_t i = threadIdx.x; i < g.heads * half / 2; i += 256) {
            const uint32_t h = i / (half / 2), e = 2 * (i % (half / 2));
            __half2 *pu = reinterpret_cast<__half2 *>(base + h * hs + e);
            __half2 *pv = reinterpret_cast<__half2 *>(base + h * hs + half + e);
            const float2 u = __half22float2(*pu), v = __half22float2(*pv), a = turn[e], b = turn[e + 1];
            *pu = __halves2half2(from_f32<__half>(u.x * a.x - v.x * a.y), from_f32<__half>(u.y * b.x - v.y * b.y));
            *pv = __halves2half2(from_f32<__half>(v.x * a.x + u.x * a.y), from_f32<__half>(v.y * b.x + u.y * b.y));
        }
        return;
    }
    for (uint32_t i = threadIdx.x; i < g.heads * half; i += 256) {
        const uint32_t h = i / half, e = i % half;
        __half *p = base + h * hs + e;
        const float u = __half2float(p[0]), v = __half2float(p[half]);
        p[0] = from_f32<__half>(u * turn[e].x - v * turn[e].y);
        p[half] = from_f32<__half>(v * turn[e].x + u * turn[e].y);
    }
}

// element pairs / quads of a weight row in either layout
__device__ __forceinline__ float2 weight2(const float *w, uint32_t k, uint32_t r, uint32_t i)
{
    if (i >= wr_ld(k)) return make_float2(0.f, 0.f);
    return *reinterpret_cast<const float2 *>(w + (size_t)r * wr_ld(k) + i);
}
__device__ __forceinline__ float2 weight2(const __half *w, uint32_t k, uint32_t r, uint32_t i)
{
    return __half22float2(*reinterpret_cast<const __half2 *>(reinterpret_cast<const char *>(w) + wr_weight_off(k, r, i)));
}
__device__ __forceinline__ float4 weight4(const float *w, uint32_t k, uint32_t r, uint32_t i)
{
    return load4(w + (size_t)r * wr_ld(k) + i);
}
__device__ __forceinline__ float4 weight4(const __half *w, uint32_t k, uint32_t r, uint32_t i)
{
    return load4(reinterpret_cast<const __half *>(reinterpret_cast<const char *>(w) + wr_weight_off(k, r, i)));
}

// A block is one head, 64 columns of the cached row and RT rows; its four warps take a quarter of the head's dimensions
// each and their sums are added in order.
template <typename TW, int RT>
__global__ void __launch_bounds__(128) latent_query_kernel(const wr_rows rw, const wr_latent_query_args a)
{
    extern __shared__ float sm_lat[];
    pdl_trigger();
    pdl_wait();
    const wr_latent_geom g = a.g;
    const uint32_t head = blockIdx.x, c0 = blockIdx.y * 64, row0 = blockIdx.z * RT, rows = min((uint32_t)RT, rw.n_rows - row0);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, hs = g.q_head();
    const float *q = a.q + ((size_t)row0 * g.heads + head) * hs;
    float *out = a.out + ((size_t)row0 * g.heads + head) * g.row();
    const size_t q_row = (size_t)g.heads * hs, out_row = (size_t)g.heads * g.row();
    if (c0 >= g.rank_pad()) {                            // the rotated part
        const uint32_t half = g.rot / 2, base = c0 - g.rank_pad();
        for (uint32_t i = threadIdx.x; i < rows * 64; i += 128) {
            const uint32_t r = i / 64, e = base + i % 64;
            float y = 0.f;
            if (e < g.rot) {
                const uint32_t row = row0 + r, p = e < half ? e : e - half;
                float sn, cs;
                angle(a.turns[p], rw.seqs[seq_of(rw, row)].pos + tok_of(rw, row), sn, cs);
                const float u = q[r * q_row + g.dim_pad() + p], v = q[r * q_row + g.dim_pad() + half + p];
                y = a.scale * (e < half ? u * cs - v * sn : v * cs + u * sn);
            }
            out[r * out_row + c0 + i % 64] = y;
        }
        return;
    }
    float *Q = sm_lat, *red = Q + RT * g.dim;            // [RT][dim], [4][RT][64]
    for (uint32_t i = threadIdx.x; i < RT * g.dim; i += 128) {
        const uint32_t r = i / g.dim;
        Q[i] = r < rows ? q[r * q_row + i % g.dim] : 0.f;
    }
    __syncthreads();
    const uint32_t per = (g.dim + 3) / 4, lo = min(warp * per, g.dim), hi = min(lo + per, g.dim);
    float acc[RT][2];
#pragma unroll
    for (int r = 0; r < RT; ++r) acc[r][0] = acc[r][1] = 0.f;
#pragma unroll 8
    for (uint32_t d = lo; d < hi; ++d) {
        const float2 w = weight2(static_cast<const TW *>(a.w_ukv), g.kv_rank, head * g.dim_pad() + d, c0 + 2 * lane);
#pragma unroll
        for (int r = 0; r < RT; ++r) {
            acc[r][0] = fmaf(Q[r * g.dim + d], w.x, acc[r][0]);
            acc[r][1] = fmaf(Q[r * g.dim + d], w.y, acc[r][1]);
        }
    }
#pragma unroll
    for (int r = 0; r < RT; ++r) {
        red[(warp * RT + r) * 64 + 2 * lane] = acc[r][0];
        red[(warp * RT + r) * 64 + 2 * lane + 1] = acc[r][1];
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < rows * 64; i += 128) {
        float y = red[i];
#pragma unroll
        for (int w = 1; w < 4; ++w) y += red[w * RT * 64 + i];
        out[i / 64 * out_row + c0 + i % 64] = a.scale * y;
    }
}

// A block is one head, 16 of its values and RT rows; a warp takes four values, its lanes the latent.
template <typename TW, typename TO, int RT>
__global__ void __launch_bounds__(128) latent_value_kernel(const wr_rows rw, const wr_latent_value_args a)
{
    extern __shared__ float sm_lat[];
    pdl_trigger();
    pdl_wait();
    const wr_latent_geom g = a.g;
    const uint32_t head = blockIdx.x, row0 = blockIdx.z * RT, rows = min((uint32_t)RT, rw.n_rows - row0), ld = wr_ld(g.kv_rank);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (uint32_t i = threadIdx.x; i < RT * ld; i += 128) {
        const uint32_t r = i / ld, c = i % ld;
        sm_lat[i] = r < rows && c < g.kv_rank ? a.o[((size_t)(row0 + r) * g.heads + head) * g.kv_rank + c] : 0.f;
    }
    __syncthreads();
#pragma unroll 1
    for (uint32_t j = 0; j < 4; ++j) {
        const uint32_t v = blockIdx.y * 16 + warp * 4 + j;
        if (v >= g.vdim) break;
        float acc[RT];
#pragma unroll
        for (int r = 0; r < RT; ++r) acc[r] = 0.f;
#pragma unroll 4
        for (uint32_t c = 4 * lane; c < ld; c += 128) {
            const float4 w = weight4(static_cast<const TW *>(a.w_ukv), g.kv_rank,
                                       g.heads * g.dim_pad() + head * g.vdim_pad() + v, c);
#pragma unroll
            for (int r = 0; r < RT; ++r) {
                const float4 o = load4(sm_lat + r * ld + c);
                acc[r] = fmaf(w.w, o.w, fmaf(w.z, o.z, fmaf(w.y, o.y, fmaf(w.x, o.x, acc[r]))));
            }
        }
        const uint32_t r = warp_reduce_many<RT>(acc, lane);
        if (reduce_writer<RT>(lane) && r < rows) Out<TO>(a.out, row0 + r, a.out_ld).put(head * g.vdim + v, acc[0]);
    }
    const uint32_t n = g.heads * g.vdim;                 // the pad columns
    if (head + 1 == g.heads && blockIdx.y + 1 == gridDim.y)
        for (uint32_t i = threadIdx.x; i < rows * (wr_ld(n) - n); i += 128)
            Out<TO>(a.out, row0 + i / (wr_ld(n) - n), a.out_ld).put(n + i % (wr_ld(n) - n), 0.f);
}

// ---- the same two steps for at most WR_CUDA_BATCH_MAX rows of a BF16 model: the rows are the M of a warp's matrix
// instruction (all sixteen always), F32 operands go in as two F16 numbers, the weights are F16 as they are stored and are
// requested before the dependency wait.

static_assert(WR_CUDA_BATCH_MAX == 16, "one matrix instruction's rows");

// A block is one head and 64 columns of the cached row, a warp 16 of them.  What leaves is the operand the attention
// kernel takes (wr_latent_split_query).
__global__ void __launch_bounds__(128) latent_query_mma_kernel(const wr_rows rw, const wr_latent_query_args a)
{
    extern __shared__ __align__(1024) uint8_t sm_mma[];
    pdl_trigger();
    const wr_latent_geom g = a.g;
    const uint32_t head = blockIdx.x, c0 = blockIdx.y * 64, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t nh = wr_latent_group(g), n = 2 * nh, hl = head % nh, hs = g.q_head();
    const size_t q_row = (size_t)g.heads * hs;
    const float *q = a.q + (size_t)head * hs;
    const float scale = a.scale * 1.4426950408889634f;
    auto operand = [&](uint32_t r) {
        return reinterpret_cast<char *>(a.out) + wr_latent_split_bytes(g) * r + (size_t)(head / nh) * (g.row() / 64) * n * 128;
    };
    auto put = [&](uint32_t r, uint32_t c, float x, float y) {          // columns c, c + 1 of row r
        uint32_t hi, lo;
        split_half2(fminf(fmaxf(x, -65504.f), 65504.f), fminf(fmaxf(y, -65504.f), 65504.f), hi, lo);
        char *out = operand(r);
        *reinterpret_cast<uint32_t *>(out + wr_latent_split_off(n, hl, c)) = hi;
        *reinterpret_cast<uint32_t *>(out + wr_latent_split_off(n, nh + hl, c)) = lo;
    };
    if (c0 >= g.rank_pad()) {                            // the rotated part
        pdl_wait();
        if (c0 > g.rank_pad()) return;                   // (one block writes all of it)
        const uint32_t half = g.rot / 2, pairs = (g.row() - c0) / 2;
        for (uint32_t i = threadIdx.x; i < rw.n_rows * pairs; i += 128) {
            const uint32_t r = i / pairs, p = i % pairs;
            float y[2] = {0.f, 0.f};
            uint32_t c[2] = {p, half + p};
            if (p < half) {
                float sn, cs;
                angle(a.turns[p], rw.seqs[seq_of(rw, r)].pos + tok_of(rw, r), sn, cs);
                const float *in = q + r * q_row + g.dim_pad();
                const float u = in[p], v = in[half + p];
                y[0] = scale * (u * cs - v * sn);
                y[1] = scale * (v * cs + u * sn);
            } else {                                     // the columns behind it are zeros
                c[0] = 2 * p;
                c[1] = 2 * p + 1;
            }
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const __half hi = from_f32<__half>(y[j]);
                char *out = operand(r);
                *reinterpret_cast<__half *>(out + wr_latent_split_off(n, hl, c0 + c[j])) = hi;
                *reinterpret_cast<__half *>(out + wr_latent_split_off(n, nh + hl, c0 + c[j])) = __float2half_rn(y[j] - __half2float(hi));
            }
        }
        return;
    }
    // weights [dim_pad][64] as stored (the head's first row is a multiple of 16: the swizzle keeps its phase)
    const uint32_t dp = g.dim_pad(), ld = dp + 8;        // (row length of the queries in shared memory)
    uint8_t *W = sm_mma;
    __half *Q = reinterpret_cast<__half *>(W + dp * 128);        // [hi | lo][16][ld]
    for (uint32_t i = threadIdx.x; i < dp * 8; i += 128) {
        const uint32_t r = i / 8, at = head * dp + r;
        const char *src = static_cast<const char *>(a.w_ukv) +
                          ((size_t)(at / kWBlock) * wr_weight_blocks(g.kv_rank) + blockIdx.y) * kWBlockBytes + at % kWBlock * 128;
        *reinterpret_cast<uint4 *>(W + r * 128 + i % 8 * 16) = *reinterpret_cast<const uint4 *>(src + i % 8 * 16);
    }
    pdl_wait();
    for (uint32_t i = threadIdx.x; i < 16 * (dp / 4); i += 128) {
        const uint32_t r = i / (dp / 4), c = 4 * (i % (dp / 4));
        const float4 v = r < rw.n_rows ? load4(q + r * q_row + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        uint32_t h0, l0, h1, l1;
        split_half2(v.x, v.y, h0, l0);
        split_half2(v.z, v.w, h1, l1);
        *reinterpret_cast<uint2 *>(Q + r * ld + c) = make_uint2(h0, h1);
        *reinterpret_cast<uint2 *>(Q + (16 + r) * ld + c) = make_uint2(l0, l1);
    }
    __syncthreads();
    float acc[2][4] = {};
    const uint32_t w_addr = smem_u32(W), q_addr = smem_u32(Q);
    for (uint32_t k0 = 0; k0 < dp; k0 += 16) {
        uint32_t hi[4], lo[4], b[4];
        // rows of the fragment: lanes 0-15 rows 0-15 at k0, lanes 16-31 the same at k0 + 8
        const uint32_t at = ((lane & 15u) * ld + k0 + (lane >> 4) * 8) * 2;
        ldmatrix_x4(hi[0], hi[1], hi[2], hi[3], q_addr + at);
        ldmatrix_x4(lo[0], lo[1], lo[2], lo[3], q_addr + 16 * ld * 2 + at);
        const uint32_t kr = k0 + (lane & 15u), piece = 2 * warp + (lane >> 4);
        ldmatrix_x4_trans(b[0], b[1], b[2], b[3], w_addr + kr * 128 + ((piece ^ (kr & 7u)) << 4));
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            mma_16816(acc[t], hi, b[2 * t], b[2 * t + 1]);
            mma_16816(acc[t], lo, b[2 * t], b[2 * t + 1]);
        }
    }
#pragma unroll
    for (int t = 0; t < 2; ++t) {
        const uint32_t c = c0 + 16 * warp + 8 * t + 2 * (lane & 3u), r = lane >> 2;
        if (r < rw.n_rows) put(r, c, acc[t][0] * scale, acc[t][1] * scale);
        if (r + 8 < rw.n_rows) put(r + 8, c, acc[t][2] * scale, acc[t][3] * scale);
    }
}

constexpr uint32_t kValueCols = 32;      // values of a block, eight per warp
constexpr uint32_t kMaxBlocks = 8;       // 64-wide blocks of a latent

// A block is one head and 32 of its values.  The attended latents come as chunks still to be added up, or finished.
__global__ void __launch_bounds__(128) latent_value_mma_kernel(const wr_rows rw, const wr_latent_value_args a)
{
    extern __shared__ __align__(1024) uint8_t sm_mma[];
    __shared__ float wt[WR_CUDA_BATCH_MAX][kLatentMaxFused];
    pdl_trigger();
    const wr_latent_geom g = a.g;
    const uint32_t head = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = lane & 3u, blocks = g.rank_pad() / 64;
    const uint32_t v0 = blockIdx.y * kValueCols + 8 * warp, row = min(v0 + (lane >> 2), g.vdim_pad() - 1);
    const uint32_t at = g.heads * g.dim_pad() + head * g.vdim_pad() + row, sw = at & 7u;
    const char *src = static_cast<const char *>(a.w_ukv) + (size_t)(at / kWBlock) * blocks * kWBlockBytes + at % kWBlock * 128;
    uint4 w[kMaxBlocks][2];
#pragma unroll
    for (uint32_t b = 0; b < kMaxBlocks; ++b)
        if (b < blocks) {
            w[b][0] = *reinterpret_cast<const uint4 *>(src + (size_t)b * kWBlockBytes + ((t ^ sw) << 4));
            w[b][1] = *reinterpret_cast<const uint4 *>(src + (size_t)b * kWBlockBytes + (((t + 4) ^ sw) << 4));
        }
    pdl_wait();
    const uint32_t rp = g.rank_pad(), ld = rp + 32;
    __half *O = reinterpret_cast<__half *>(sm_mma);      // [hi | lo][16][ld]
    const float *ml = a.ml;
    if (ml) {
        for (uint32_t r = warp; r < rw.n_rows; r += 4)
            latent_chunk_weights(ml + ((size_t)r * g.heads + head) * a.chunks * 2, a.lens.count[r], wt[r], lane);
        __syncthreads();
    }
    for (uint32_t i = threadIdx.x; i < 16 * (rp / 4); i += 128) {
        const uint32_t r = i / (rp / 4), c = 4 * (i % (rp / 4));
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        if (r < rw.n_rows) {
            const float *in = a.o + ((size_t)r * g.heads + head) * (ml ? a.chunks : 1u) * rp + c;
            o = ml ? latent_chunk_sum(in, rp, wt[r], a.lens.count[r]) : load4(in);
        }
        uint32_t h0, l0, h1, l1;
        split_half2(o.x, o.y, h0, l0);
        split_half2(o.z, o.w, h1, l1);
        *reinterpret_cast<uint2 *>(O + r * ld + c) = make_uint2(h0, h1);
        *reinterpret_cast<uint2 *>(O + (16 + r) * ld + c) = make_uint2(l0, l1);
    }
    __syncthreads();
    // The order of the latent in the sum is the weights' own: a lane's 16-byte piece is two steps of its fragment.
    float acc[4] = {}, acc_l[4] = {}, acc2[4] = {}, acc2_l[4] = {};      // (four chains of products)
    const __half *lo_rows = O + 16 * ld;
#pragma unroll
    for (uint32_t b = 0; b < kMaxBlocks; ++b)
        if (b < blocks) {
#pragma unroll
            for (uint32_t p = 0; p < 2; ++p) {
                const uint32_t c = 64 * b + 8 * (t + 4 * p), r = lane >> 2;
                const uint4 h0 = *reinterpret_cast<const uint4 *>(O + r * ld + c), h1 = *reinterpret_cast<const uint4 *>(O + (r + 8) * ld + c);
                const uint4 l0 = *reinterpret_cast<const uint4 *>(lo_rows + r * ld + c);
                const uint4 l1 = *reinterpret_cast<const uint4 *>(lo_rows + (r + 8) * ld + c);
                const uint32_t ah[2][4] = {{h0.x, h1.x, h0.y, h1.y}, {h0.z, h1.z, h0.w, h1.w}};
                const uint32_t al[2][4] = {{l0.x, l1.x, l0.y, l1.y}, {l0.z, l1.z, l0.w, l1.w}};
                mma_16816(acc, ah[0], w[b][p].x, w[b][p].y);
                mma_16816(acc_l, al[0], w[b][p].x, w[b][p].y);
                mma_16816(acc2, ah[1], w[b][p].z, w[b][p].w);
                mma_16816(acc2_l, al[1], w[b][p].z, w[b][p].w);
            }
        }
#pragma unroll
    for (uint32_t j = 0; j < 4; ++j) {
        const uint32_t r = (lane >> 2) + 8 * (j >> 1), v = v0 + 2 * t + (j & 1u);
        if (r < rw.n_rows && v < g.vdim) Out<Split>(a.out, r, a.out_ld).put(head * g.vdim + v, (acc[j] + acc2[j]) + (acc_l[j] + acc2_l[j]));
    }
    const uint32_t n = g.heads * g.vdim, pad = wr_ld(n) - n;
    if (head + 1 == g.heads && blockIdx.y + 1 == gridDim.y)
        for (uint32_t i = threadIdx.x; i < rw.n_rows * pad; i += 128) Out<Split>(a.out, i / pad, a.out_ld).put(n + i % pad, 0.f);
}

template <typename TW, int RT> int query_rows(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_query_args &a)
{
    const size_t smem = (size_t)(RT * a.g.dim + 4 * RT * 64) * 4;
    const int rc = allow_smem(latent_query_kernel<TW, RT>, smem);
    if (rc != WR_CUDA_OK) return rc;
    WR_CUDA_TRY(wr_launch_pdl(latent_query_kernel<TW, RT>, dim3(a.g.heads, a.g.row() / 64, (rw.n_rows + RT - 1) / RT), dim3(128),
                              smem, ctx->stream, rw, a));
    return finish_launch(ctx);
}
template <typename TW> int query_any(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_query_args &a)
{
    if (rw.n_rows == 1) return query_rows<TW, 1>(ctx, rw, a);
    if (rw.n_rows <= 4) return query_rows<TW, 4>(ctx, rw, a);
    return query_rows<TW, kTileRows>(ctx, rw, a);
}

template <typename TW, typename TO, int RT> int value_rows(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_value_args &a)
{
    const size_t smem = (size_t)RT * wr_ld(a.g.kv_rank) * 4;
    const int rc = allow_smem(latent_value_kernel<TW, TO, RT>, smem);
    if (rc != WR_CUDA_OK) return rc;
    WR_CUDA_TRY(wr_launch_pdl(latent_value_kernel<TW, TO, RT>, dim3(a.g.heads, (a.g.vdim + 15) / 16, (rw.n_rows + RT - 1) / RT),
                              dim3(128), smem, ctx->stream, rw, a));
    return finish_launch(ctx);
}
template <typename TW, typename TO> int value_any(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_value_args &a)
{
    if (rw.n_rows == 1) return value_rows<TW, TO, 1>(ctx, rw, a);
    if (rw.n_rows <= 4) return value_rows<TW, TO, 4>(ctx, rw, a);
    return value_rows<TW, TO, kTileRows>(ctx, rw, a);
}

}  // namespace

int wr_latent_prep_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_prep_args &a)
{
    const dim3 grid(rw.n_rows, (a.own ? 2 : 1) + (a.route ? 1 : 0));
    const dim3 block(rw.n_rows <= WR_CUDA_BATCH_MAX ? kPrepThreads : kPrepThreads / 2);
    const wr_route_args route = a.route ? *a.route : wr_route_args{};
    const size_t smem = !a.route ? 0 : route.tile ? (size_t)route.experts * 4 : route_few_smem(route);
    auto launch = [&](auto kernel) {
        const int rc = allow_smem(kernel, smem);
        if (rc != WR_CUDA_OK) return rc;
        WR_CUDA_TRY(wr_launch_pdl(kernel, grid, block, smem, ctx->stream, rw, a, route));
        return finish_launch(ctx);
    };
    if (a.cq_type == WR_ACT_BF16) return launch(latent_prep_kernel<__nv_bfloat16>);
    if (a.cq_type == WR_ACT_SPLIT) return launch(latent_prep_kernel<Split>);
    return launch(latent_prep_kernel<float>);
}

int wr_latent_rotate_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_geom &g, const double *turns, void *q)
{
    WR_CUDA_TRY(wr_launch_pdl(latent_rotate_kernel, dim3(rw.n_rows), dim3(256), 0, ctx->stream, rw, g, turns, static_cast<__half *>(q)));
    return finish_launch(ctx);
}

int wr_latent_query_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_query_args &a)
{
    if (a.split) {
        const size_t smem = (size_t)a.g.dim_pad() * 128 + 2 * 16 * (a.g.dim_pad() + 8) * 2;
        const int rc = allow_smem(latent_query_mma_kernel, smem);
        if (rc != WR_CUDA_OK) return rc;
        WR_CUDA_TRY(wr_launch_pdl(latent_query_mma_kernel, dim3(a.g.heads, a.g.row() / 64), dim3(128), smem, ctx->stream, rw, a));
        return finish_launch(ctx);
    }
    return a.w_type == WR_ACT_F16 ? query_any<__half>(ctx, rw, a) : query_any<float>(ctx, rw, a);
}

int wr_latent_value_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_value_args &a)
{
    if (a.split) {
        const size_t smem = (size_t)2 * 16 * (a.g.rank_pad() + 32) * 2;
        const int rc = allow_smem(latent_value_mma_kernel, smem);
        if (rc != WR_CUDA_OK) return rc;
        WR_CUDA_TRY(wr_launch_pdl(latent_value_mma_kernel, dim3(a.g.heads, (a.g.vdim + kValueCols - 1) / kValueCols), dim3(128), smem,
                                  ctx->stream, rw, a));
        return finish_launch(ctx);
    }
    if (a.w_type == WR_ACT_F32) return value_any<float, float>(ctx, rw, a);
    return a.out_type == WR_ACT_SPLIT ? value_any<__half, Split>(ctx, rw, a) : value_any<__half, __nv_bfloat16>(ctx, rw, a);
}
