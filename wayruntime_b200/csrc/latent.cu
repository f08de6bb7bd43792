// latent.cu — what surrounds attention over a shared latent row: norms and rotation of the projection, queries moved
// into the latent's space, and the attended latent turned back into values.
//
// All arithmetic is F32 (angles reduced in double).  A row's result depends on its session alone; the sums of an
// output follow one order whatever the number of rows.
#include <algorithm>

#include "gemm_bf16.cuh"
#include "rows_dev.cuh"
#include "warp_reduce.cuh"

namespace {

constexpr uint32_t kPrepThreads = 256, kTileRows = 16;

__device__ __forceinline__ void angle(double turns, uint32_t pos, float &sn, float &cs)
{
    const double a = turns * (double)pos;                // in turns, reduced before it leaves double
    sincospif(2.0f * (float)(a - rint(a)), &sn, &cs);
}

// grid.y 0: the query latent; 1: the session's row
template <typename TO>
__global__ void __launch_bounds__(kPrepThreads) latent_prep_kernel(const wr_rows rw, const wr_latent_prep_args a)
{
    __shared__ float part[kPrepThreads / 32];
    pdl_trigger();
    pdl_wait();
    const uint32_t row = blockIdx.x, n = blockIdx.y ? a.g.kv_rank : a.g.q_rank;
    const float *in = a.in + (size_t)row * a.ld, *x = in + (blockIdx.y ? a.c_off : 0u);
    const float *w = blockIdx.y ? a.c_norm : a.q_norm;
    float ss = 0.f;
    for (uint32_t i = threadIdx.x; i < n; i += kPrepThreads) ss = fmaf(x[i], x[i], ss);
    const float inv = 1.0f / sqrtf(block_sum<kPrepThreads / 32>(ss, part) / (float)n + a.eps);
    if (blockIdx.y == 0) {
        const Out<TO> out(a.cq, row, wr_ld(n));
        for (uint32_t i = threadIdx.x; i < wr_ld(n); i += kPrepThreads) out.put(i, i < n ? x[i] * inv * w[i] : 0.f);
        return;
    }
    const wr_seq_dev s = rw.seqs[seq_of(rw, row)];
    const uint32_t pos = s.pos + tok_of(rw, row), tok = pos % kPageTokens, half = a.g.rot / 2;
    char *page = reinterpret_cast<char *>(s.pages[(size_t)a.layer * s.n_pages + pos / kPageTokens]);
    auto put = [&](uint32_t d, float v) {
        char *p = page + wr_geom_off(a.kv, 0, 0, tok, d);
        if (a.kv.elem == WR_CUDA_F32) *reinterpret_cast<float *>(p) = v;
        else *reinterpret_cast<__half *>(p) = from_f32<__half>(v);
    };
    for (uint32_t i = threadIdx.x; i < n; i += kPrepThreads) put(i, x[i] * inv * w[i]);
    const float *r = in + a.r_off;
    for (uint32_t i = threadIdx.x; i < half; i += kPrepThreads) {
        float sn, cs;
        angle(a.turns[i], pos, sn, cs);
        const float u = r[i], v = r[i + half];
        put(a.g.rank_pad() + i, u * cs - v * sn);
        put(a.g.rank_pad() + half + i, v * cs + u * sn);
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
    const dim3 grid(rw.n_rows, a.own ? 2 : 1), block(kPrepThreads);
    if (a.cq_type == WR_ACT_BF16) WR_CUDA_TRY(wr_launch_pdl(latent_prep_kernel<__nv_bfloat16>, grid, block, 0, ctx->stream, rw, a));
    else if (a.cq_type == WR_ACT_SPLIT) WR_CUDA_TRY(wr_launch_pdl(latent_prep_kernel<Split>, grid, block, 0, ctx->stream, rw, a));
    else WR_CUDA_TRY(wr_launch_pdl(latent_prep_kernel<float>, grid, block, 0, ctx->stream, rw, a));
    return finish_launch(ctx);
}

int wr_latent_rotate_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_geom &g, const double *turns, void *q)
{
    WR_CUDA_TRY(wr_launch_pdl(latent_rotate_kernel, dim3(rw.n_rows), dim3(256), 0, ctx->stream, rw, g, turns, static_cast<__half *>(q)));
    return finish_launch(ctx);
}

int wr_latent_query_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_query_args &a)
{
    return a.w_type == WR_ACT_F16 ? query_any<__half>(ctx, rw, a) : query_any<float>(ctx, rw, a);
}

int wr_latent_value_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_value_args &a)
{
    if (a.w_type == WR_ACT_F32) return value_any<float, float>(ctx, rw, a);
    return a.out_type == WR_ACT_SPLIT ? value_any<__half, Split>(ctx, rw, a) : value_any<__half, __nv_bfloat16>(ctx, rw, a);
}
