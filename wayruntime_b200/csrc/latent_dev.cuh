// latent_dev.cuh — how chunks of attended latents are added up (latent.cu, attn_latent.cu): one arithmetic for both.
#pragma once

#include "rows_dev.cuh"

#ifdef __CUDACC__
namespace {

constexpr uint32_t kLatentMaxFused = 16;  // chunks of a row that the value kernel adds up itself

// One warp: weights of a row and head's n chunks out of their (maximum, sum) pairs, divided by the whole sum.
__device__ __forceinline__ void latent_chunk_weights(const float *ml, uint32_t n, float *w, uint32_t lane)
{
    float m = -INFINITY, l = 0.f;
    for (uint32_t i = lane; i < n; i += 32) m = fmaxf(m, ml[2 * i]);
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    for (uint32_t i = lane; i < n; i += 32) {
        const float e = expf(ml[2 * i] - m);
        w[i] = e;
        l = fmaf(e, ml[2 * i + 1], l);
    }
    l = warp_sum(l);
    __syncwarp();
    for (uint32_t i = lane; i < n; i += 32) w[i] = __fdiv_rn(w[i], l);
}

// Four columns of the chunks (ld floats apart), in order.
__device__ __forceinline__ float4 latent_chunk_sum(const float *in, uint32_t ld, const float *w, uint32_t n)
{
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    uint32_t i = 0;
    for (; i + 4 <= n; i += 4) {
        float4 v[4];
#pragma unroll
        for (uint32_t j = 0; j < 4; ++j) v[j] = load4(in + (size_t)(i + j) * ld);
#pragma unroll
        for (uint32_t j = 0; j < 4; ++j)
            s = make_float4(fmaf(w[i + j], v[j].x, s.x), fmaf(w[i + j], v[j].y, s.y), fmaf(w[i + j], v[j].z, s.z),
                            fmaf(w[i + j], v[j].w, s.w));
    }
    for (; i < n; ++i) {
        const float4 v = load4(in + (size_t)i * ld);
        s = make_float4(fmaf(w[i], v.x, s.x), fmaf(w[i], v.y, s.y), fmaf(w[i], v.z, s.z), fmaf(w[i], v.w, s.w));
    }
    return s;
}

}  // namespace
#endif
