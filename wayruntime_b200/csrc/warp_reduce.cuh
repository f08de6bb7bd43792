// warp_reduce.cuh — many sums across a warp at once.
#pragma once

#include <stdint.h>

#ifdef __CUDACC__
namespace {

// Sum M per-lane partials across the warp.  Afterwards every lane holds, in
// v[0], the warp total of the value whose index the function returns; lanes
// whose index bits agree hold the same total.  Each step that still has more
// than one live value halves them by exchanging the half the partner keeps,
// so the whole reduction costs about M shuffles instead of 5*M.
template <int M>
__device__ __forceinline__ int warp_reduce_many(float (&v)[M], int lane)
{
    static_assert(M >= 1 && M <= 32 && (M & (M - 1)) == 0, "power of two up to 32");
    int width = M, idx = 0;
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) {
        if (width > 1) {
            const int half = width / 2;
            const bool upper = (lane & o) != 0;
#pragma unroll
            for (int i = 0; i < M / 2; ++i) {
                if (i < half) {
                    const float send = upper ? v[i] : v[i + half];
                    const float keep = upper ? v[i + half] : v[i];
                    v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
            }
            if (upper) idx += half;
            width = half;
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
        }
    }
    return idx;
}

// lanes that write: those whose non-index bits are zero
template <int M>
__device__ __forceinline__ bool reduce_writer(int lane)
{
    // index bits are the top log2(M) of the five lane bits
    int used = 0;
    for (int m = M, o = 16; m > 1; m >>= 1, o >>= 1) used |= o;
    return (lane & ~used & 31) == 0;
}

}  // namespace
#endif
