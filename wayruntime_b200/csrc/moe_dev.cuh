// moe_dev.cuh — the choice of experts, for kernels that have a row's logits at hand (moe.cu, latent.cu).
#pragma once

#include "rows_dev.cuh"

#ifdef __CUDACC__
namespace {

// One warp's row: z (shared memory, experts values) loses the chosen logits.
__device__ __forceinline__ void choose(float *z, const wr_route_args &a, uint32_t row)
{
    const uint32_t lane = threadIdx.x & 31;
    const float *in = a.logits + (size_t)row * a.ld;
    for (uint32_t e = lane; e < a.experts; e += 32) z[e] = in[e] + a.bias[e];
    __syncwarp();
    float first = 0.f, sum = 0.f;
    for (uint32_t s = 0; s < a.top; ++s) {
        float best = -INFINITY;
        uint32_t at = ~0u;
        for (uint32_t e = lane; e < a.experts; e += 32)
            if (z[e] > best || at == ~0u) {
                best = z[e];
                at = e;
            }
#pragma unroll
        for (int o = 16; o >= 1; o >>= 1) {
            const float b = __shfl_xor_sync(0xffffffffu, best, o);
            const uint32_t t = __shfl_xor_sync(0xffffffffu, at, o);
            if (t != ~0u && (at == ~0u || b > best || (b == best && t < at))) {
                best = b;
                at = t;
            }
        }
        if (s == 0) first = best;
        const float w = expf(best - first);
        sum += w;
        if (lane == 0) {
            a.expert[(size_t)row * a.top + s] = at;
            a.weight[(size_t)row * a.top + s] = w;
            z[at] = -INFINITY;
        }
        __syncwarp();
    }
    for (uint32_t s = lane; s < a.top; s += 32) a.weight[(size_t)row * a.top + s] /= sum;
}

// One block, all of a step's few rows: their choices, then the list of the experts in use, in ascending order.
// sm: (WR_CUDA_BATCH_MAX + 1) * experts words.
__device__ __forceinline__ void route_few(float *sm, const wr_route_args &a, uint32_t rows)
{
    const uint32_t warp = threadIdx.x >> 5, warps = blockDim.x >> 5, lane = threadIdx.x & 31;
    for (uint32_t r = warp; r < rows; r += warps) choose(sm + r * a.experts, a, r);
    uint32_t *number = reinterpret_cast<uint32_t *>(sm + WR_CUDA_BATCH_MAX * a.experts);
    for (uint32_t e = threadIdx.x; e < a.experts; e += blockDim.x) number[e] = 0;
    __syncthreads();
    const uint32_t pairs = rows * a.top;
    for (uint32_t i = threadIdx.x; i < pairs; i += blockDim.x) number[a.expert[i]] = 1;
    __syncthreads();
    if (warp == 0) {
        uint32_t used = 0;
        for (uint32_t e0 = 0; e0 < a.experts; e0 += 32) {
            const uint32_t e = e0 + lane;
            const bool in = e < a.experts && number[e];
            const uint32_t votes = __ballot_sync(0xffffffffu, in), at = used + __popc(votes & ((1u << lane) - 1u));
            if (in) {
                number[e] = at;
                a.list[at] = e;
            }
            used += __popc(votes);
        }
        if (lane == 0) *a.count = used;
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < pairs; i += blockDim.x) a.place[i] = number[a.expert[i]];
}
inline size_t route_few_smem(const wr_route_args &a) { return (size_t)(WR_CUDA_BATCH_MAX + 1) * a.experts * 4; }

}  // namespace
#endif
