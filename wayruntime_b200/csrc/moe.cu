// moe.cu — routing of rows to experts, and what surrounds the experts' products.
//
// Logits, choice and weights are F32; of equal logits the lower expert wins.  A row's result depends on the row alone:
// places only say where its inputs and outputs lie, and its slots are added up in order.
#include <algorithm>

#include "gemm_bf16.cuh"
#include "moe_dev.cuh"

namespace {

constexpr uint32_t kSortThreads = 1024;

constexpr uint32_t kRouteWarps = 8;

__global__ void __launch_bounds__(kRouteWarps * 32) moe_choose_kernel(const wr_rows rw, const wr_route_args a)
{
    extern __shared__ float sm_moe[];
    pdl_trigger();
    pdl_wait();
    const uint32_t row = blockIdx.x * kRouteWarps + (threadIdx.x >> 5);
    if (row < rw.n_rows) choose(sm_moe + (threadIdx.x >> 5) * a.experts, a, row);
}

__global__ void __launch_bounds__(WR_CUDA_BATCH_MAX * 32) moe_route_few_kernel(const wr_rows rw, const wr_route_args a)
{
    extern __shared__ float sm_moe[];
    pdl_trigger();
    pdl_wait();
    route_few(sm_moe, a, rw.n_rows);
}

// Many rows: places by expert, every expert's from a multiple of the tile on.
__global__ void __launch_bounds__(kSortThreads) moe_sort_kernel(const wr_rows rw, const wr_route_args a)
{
    extern __shared__ uint32_t sm_sort[];
    uint32_t *n = sm_sort, *next = n + a.experts;        // pairs per expert; the next free place
    pdl_trigger();
    pdl_wait();
    const uint32_t pairs = rw.n_rows * a.top, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (uint32_t e = threadIdx.x; e < a.experts; e += kSortThreads) n[e] = 0;
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < pairs; i += kSortThreads) atomicAdd(&n[a.expert[i]], 1u);
    __syncthreads();
    if (warp == 0) {
        uint32_t tiles = 0;
        for (uint32_t e0 = 0; e0 < a.experts; e0 += 32) {
            const uint32_t e = e0 + lane, mine = e < a.experts ? (n[e] + a.tile - 1) / a.tile : 0u;
            uint32_t upto = mine;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const uint32_t v = __shfl_up_sync(0xffffffffu, upto, o);
                if (lane >= (uint32_t)o) upto += v;
            }
            if (e < a.experts) next[e] = (tiles + upto - mine) * a.tile;
            tiles += __shfl_sync(0xffffffffu, upto, 31);
        }
        if (lane == 0) *a.count = tiles;
    }
    __syncthreads();
    for (uint32_t e = warp; e < a.experts; e += kSortThreads / 32) {
        const uint32_t first = next[e], last = first + (n[e] + a.tile - 1) / a.tile * a.tile;
        for (uint32_t t = first + lane * a.tile; t < last; t += 32 * a.tile) a.list[t / a.tile] = e;
        for (uint32_t p = first + n[e] + lane; p < last; p += 32) a.row_of[p] = ~0u;
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < pairs; i += kSortThreads) {
        const uint32_t p = atomicAdd(&next[a.expert[i]], 1u);
        a.place[i] = p;
        a.row_of[p] = i / a.top;
    }
}

__global__ void __launch_bounds__(256) moe_gather_kernel(const uint4 *x, uint4 *out, uint32_t vecs, const uint32_t *row_of,
                                                         const uint32_t *count, uint32_t tile)
{
    pdl_trigger();
    pdl_wait();
    const uint32_t p = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (p >= *count * tile) return;
    const uint32_t row = row_of[p];
    if (row == ~0u) return;
    for (uint32_t i = threadIdx.x & 31; i < vecs; i += 32) out[(size_t)p * vecs + i] = x[(size_t)row * vecs + i];
}

template <typename T> __global__ void __launch_bounds__(256) moe_combine_kernel(const wr_rows rw, const wr_combine_args a)
{
    pdl_trigger();
    pdl_wait();
    const uint32_t row = blockIdx.x, c = 4 * (blockIdx.y * 256 + threadIdx.x);
    if (c >= a.width) return;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (uint32_t k = 0; k < a.top; ++k) {
        const uint32_t p = a.place[(size_t)row * a.top + k];
        const float w = a.weight[(size_t)row * a.top + k];
        const size_t at = a.few ? (size_t)WR_CUDA_BATCH_MAX * p + row : p;
        const float4 y = load4(static_cast<const T *>(a.y) + at * a.ld + c);
        s = make_float4(fmaf(w, y.x, s.x), fmaf(w, y.y, s.y), fmaf(w, y.z, s.z), fmaf(w, y.w, s.w));
    }
    float *r = a.resid + (size_t)row * a.ld + c;
    float4 x = load4(r);
    x.x = fmaf(a.mul, s.x, x.x);
    if (c + 1 < a.width) x.y = fmaf(a.mul, s.y, x.y);
    if (c + 2 < a.width) x.z = fmaf(a.mul, s.z, x.z);
    if (c + 3 < a.width) x.w = fmaf(a.mul, s.w, x.w);
    store4(r, x);
}

// 32 places x 32 output columns of one expert; a thread has four places of one column.
template <bool PAIR> __global__ void __launch_bounds__(256) moe_f32_kernel(const wr_moe_f32_args a)
{
    constexpr uint32_t kT = kMoeTileF32;
    __shared__ float xs[kT][kT + 1], wg[kT][kT + 1], wu[PAIR ? kT : 1][kT + 1];
    pdl_trigger();
    pdl_wait();
    if (blockIdx.y >= *a.count) return;
    const uint32_t e = a.list[blockIdx.y], p0 = blockIdx.y * kT, n0 = blockIdx.x * kT, ldk = wr_ld(a.k);
    const uint32_t col = threadIdx.x & 31, r0 = (threadIdx.x >> 5) * 4;
    const float *gate = a.gate + e * a.stride, *up = PAIR ? a.up + e * a.stride : nullptr;
    float g[4] = {0.f, 0.f, 0.f, 0.f}, u[4] = {0.f, 0.f, 0.f, 0.f};
    for (uint32_t k0 = 0; k0 < a.k; k0 += kT) {
        __syncthreads();
        for (uint32_t i = threadIdx.x; i < kT * kT; i += 256) {
            const uint32_t r = i / kT, k = i % kT, n = n0 + r;
            const uint32_t row = a.row_of ? a.row_of[p0 + r] : p0 + r;
            const bool in = k0 + k < a.k;
            xs[r][k] = in && row != ~0u ? a.x[(size_t)row * a.x_ld + k0 + k] : 0.f;
            wg[r][k] = in && n < a.n ? gate[(size_t)n * ldk + k0 + k] : 0.f;
            if (PAIR) wu[r][k] = in && n < a.n ? up[(size_t)n * ldk + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (uint32_t k = 0; k < kT; ++k)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                g[j] = fmaf(xs[r0 + j][k], wg[col][k], g[j]);
                if (PAIR) u[j] = fmaf(xs[r0 + j][k], wu[PAIR ? col : 0][k], u[j]);
            }
    }
    if (n0 + col >= a.out_ld) return;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        float y = g[j];
        if (PAIR) {
            const float gg = fminf(g[j], a.limit), uu = fminf(fmaxf(u[j], -a.limit), a.limit);
            y = gg / (1.0f + expf(-a.alpha * gg)) * (uu + 1.0f);
        }
        a.out[(size_t)(p0 + r0 + j) * a.out_ld + n0 + col] = n0 + col < a.n ? y : 0.f;
    }
}

}  // namespace

int wr_route_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_route_args &a)
{
    if (!a.tile) {
        if (a.chosen) return WR_CUDA_OK;
        const size_t smem = route_few_smem(a);
        const int rc = allow_smem(moe_route_few_kernel, smem);
        if (rc != WR_CUDA_OK) return rc;
        WR_CUDA_TRY(wr_launch_pdl(moe_route_few_kernel, dim3(1), dim3(WR_CUDA_BATCH_MAX * 32), smem, ctx->stream, rw, a));
        return finish_launch(ctx);
    }
    size_t smem = (size_t)kRouteWarps * a.experts * 4;
    int rc = allow_smem(moe_choose_kernel, smem);
    if (rc != WR_CUDA_OK) return rc;
    if (!a.chosen) {
        WR_CUDA_TRY(wr_launch_pdl(moe_choose_kernel, dim3((rw.n_rows + kRouteWarps - 1) / kRouteWarps), dim3(kRouteWarps * 32),
                                  smem, ctx->stream, rw, a));
        rc = finish_launch(ctx);
        if (rc != WR_CUDA_OK) return rc;
    }
    smem = (size_t)2 * a.experts * 4;
    rc = allow_smem(moe_sort_kernel, smem);
    if (rc != WR_CUDA_OK) return rc;
    WR_CUDA_TRY(wr_launch_pdl(moe_sort_kernel, dim3(1), dim3(kSortThreads), smem, ctx->stream, rw, a));
    return finish_launch(ctx);
}

int wr_moe_gather_launch(wr_cuda_ctx *ctx, const void *x, void *out, uint32_t ld, const uint32_t *row_of,
                         const uint32_t *count, uint32_t max_tiles, uint32_t tile)
{
    WR_CUDA_TRY(wr_launch_pdl(moe_gather_kernel, dim3((max_tiles * tile + 7) / 8), dim3(256), 0, ctx->stream,
                              static_cast<const uint4 *>(x), static_cast<uint4 *>(out), ld / 8, row_of, count, tile));
    return finish_launch(ctx);
}

int wr_moe_combine_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_combine_args &a)
{
    const dim3 grid(rw.n_rows, (a.width + 1023) / 1024), block(256);
    if (a.type == WR_ACT_BF16) WR_CUDA_TRY(wr_launch_pdl(moe_combine_kernel<__nv_bfloat16>, grid, block, 0, ctx->stream, rw, a));
    else WR_CUDA_TRY(wr_launch_pdl(moe_combine_kernel<float>, grid, block, 0, ctx->stream, rw, a));
    return finish_launch(ctx);
}

int wr_moe_f32_launch(wr_cuda_ctx *ctx, const wr_moe_f32_args &a)
{
    const dim3 grid((a.out_ld + kMoeTileF32 - 1) / kMoeTileF32, a.max_tiles), block(256);
    if (a.up) WR_CUDA_TRY(wr_launch_pdl(moe_f32_kernel<true>, grid, block, 0, ctx->stream, a));
    else WR_CUDA_TRY(wr_launch_pdl(moe_f32_kernel<false>, grid, block, 0, ctx->stream, a));
    return finish_launch(ctx);
}
