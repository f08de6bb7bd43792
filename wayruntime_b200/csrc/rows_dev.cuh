// rows_dev.cuh — device helpers of the row kernels: element types, vector loads and stores, where a row goes.
#pragma once

#include <cuda_bf16.h>

#include "mixers.cuh"

#ifdef __CUDACC__
namespace {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f32(__half v) { return __half2float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
template <> __device__ __forceinline__ __half from_f32<__half>(float v)
{
    return __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f));
}
// (a few units in the last place: the exponential and the quotient are the short sequences)
__device__ __forceinline__ float sigmoidf(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }
__device__ __forceinline__ float siluf(float x) { return __fdividef(x, 1.0f + __expf(-x)); }

// two F32 values in one 64-bit register: one issue slot for two elements
__device__ __forceinline__ uint64_t pack2(float a, float b)
{
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void unpack2(uint64_t v, float &a, float &b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c)
{
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b)
{
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

// four / eight consecutive values (addresses aligned to the vector)
__device__ __forceinline__ float4 load4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16 *p)
{
    const uint2 u = *reinterpret_cast<const uint2 *>(p);
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                       __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ float4 load4(const __half *p)
{
    const uint2 u = *reinterpret_cast<const uint2 *>(p);
    const float2 a = __half22float2(*reinterpret_cast<const __half2 *>(&u.x)), b = __half22float2(*reinterpret_cast<const __half2 *>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16 *p, float4 v)
{
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
}
template <typename T> __device__ __forceinline__ void load8v(const T *p, float (&v)[8])
{
    const float4 a = load4(p), b = load4(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void load8v(const __nv_bfloat16 *p, float (&v)[8])
{
    const uint4 u = *reinterpret_cast<const uint4 *>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        v[2 * i] = __uint_as_float(w[i] << 16);
        v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
template <typename T> __device__ __forceinline__ void store8v(T *p, const float (&v)[8])
{
    store4(p, make_float4(v[0], v[1], v[2], v[3]));
    store4(p + 4, make_float4(v[4], v[5], v[6], v[7]));
}
__device__ __forceinline__ void store8v(__nv_bfloat16 *p, const float (&v)[8])
{
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        w[i] = *reinterpret_cast<const uint32_t *>(&h);
    }
    *reinterpret_cast<uint4 *>(p) = make_uint4(w[0], w[1], w[2], w[3]);
}
__device__ __forceinline__ void store8v(__half *p, const float (&v)[8])
{
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const __half2 h = __halves2half2(from_f32<__half>(v[2 * i]), from_f32<__half>(v[2 * i + 1]));
        w[i] = *reinterpret_cast<const uint32_t *>(&h);
    }
    *reinterpret_cast<uint4 *>(p) = make_uint4(w[0], w[1], w[2], w[3]);
}

// Where a kernel leaves its rows: plain ones of type T, or (Split) F32 values as two BF16 numbers, the second
// WR_CUDA_BATCH_MAX rows behind the first.
struct Split {};
template <typename T> struct Out {
    T *p;
    __device__ __forceinline__ Out(void *base, uint32_t row, uint32_t ld) : p(static_cast<T *>(base) + (size_t)row * ld) {}
    __device__ __forceinline__ void put(uint32_t i, float v) const { p[i] = from_f32<T>(v); }
    __device__ __forceinline__ void put4(uint32_t i, float4 v) const { store4(p + i, v); }
    __device__ __forceinline__ void put8(uint32_t i, const float (&v)[8]) const { store8v(p + i, v); }
};
template <> struct Out<Split> {
    __nv_bfloat16 *p;
    size_t lo;
    __device__ __forceinline__ Out(void *base, uint32_t row, uint32_t ld)
        : p(static_cast<__nv_bfloat16 *>(base) + (size_t)row * ld), lo((size_t)WR_CUDA_BATCH_MAX * ld) {}
    static __device__ __forceinline__ float rest(float v) { return v - __bfloat162float(__float2bfloat16_rn(v)); }
    __device__ __forceinline__ void put(uint32_t i, float v) const
    {
        p[i] = __float2bfloat16_rn(v);
        p[lo + i] = __float2bfloat16_rn(rest(v));
    }
    __device__ __forceinline__ void put4(uint32_t i, float4 v) const
    {
        store4(p + i, v);
        store4(p + lo + i, make_float4(rest(v.x), rest(v.y), rest(v.z), rest(v.w)));
    }
    __device__ __forceinline__ void put8(uint32_t i, const float (&v)[8]) const
    {
        float r[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) r[e] = rest(v[e]);
        store8v(p + i, v);
        store8v(p + lo + i, r);
    }
};

// the session of a row and the row's place among the session's tokens of this step
__device__ __forceinline__ uint32_t seq_of(const wr_rows &rw, uint32_t row) { return rw.decode ? row : 0u; }
__device__ __forceinline__ uint32_t tok_of(const wr_rows &rw, uint32_t row) { return rw.decode ? 0u : row; }
__device__ __forceinline__ uint32_t row0_of(const wr_rows &rw, uint32_t seq) { return rw.decode ? seq : 0u; }

__device__ __forceinline__ float warp_sum(float v)
{
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// the whole block's sum, warps in order; part: a float per warp
__device__ __forceinline__ float block_sum(float v, float *part)
{
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    for (uint32_t i = 0; i < blockDim.x >> 5; ++i) t += part[i];
    return t;
}

inline int finish_launch(wr_cuda_ctx *ctx)
{
    ctx->launches++;
    WR_CUDA_TRY(cudaGetLastError());
    return WR_CUDA_OK;
}

template <typename K> int allow_smem(K k, size_t smem)
{
    if (smem > 227 * 1024) return WR_CUDA_ERR_LIMIT;
    if (smem > 48 * 1024)
        WR_CUDA_TRY(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return WR_CUDA_OK;
}

}  // namespace
#endif
