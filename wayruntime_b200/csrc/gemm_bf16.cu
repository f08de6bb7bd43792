// gemm_bf16.cu — out[m][n] = act(x . w^T + bias) + add on the 5th-generation tensor cores.
//
// Persistent CTAs (one per SM) walk output tiles of 128 rows x BN columns, m fastest so that the
// tiles in flight share weight rows in L2.  Warp 0 feeds a ring of shared-memory stages with TMA
// (64 K-values of both operands per stage: activations through a tensor map, weights as linear copies
// of blocks stored in the operand's layout; what lies beyond K arrives as zeros), warp 1 issues tcgen05.mma into one of two TMEM accumulators, warps 2-5 read the other one
// back and write the finished rows (bias, softplus, residual; F32, BF16 or saturated F16), so that a
// tile's output overlaps the next tile's products.  Columns may be gate / up pairs, of which the activation leaves
// (wr_pair_args), row tiles may have weights of their own (wr_group_args), and activations may come from a cache's pages.  Every wait is bounded by the context's wait
// limit; a warp that gives up records an error word and all of them leave.
#include <cuda_bf16.h>

#include <algorithm>

#include "gemm_bf16.cuh"
#include "tcgen05_dev.cuh"

namespace {

constexpr uint32_t kBM = 128, kBK = 64;
constexpr uint32_t kThreads = 192;
constexpr uint32_t kABytes = kBM * kBK * 2;
constexpr uint32_t kStageBudget = 196608;

template <uint32_t BN> struct Tile {
    static constexpr uint32_t kBBytes = BN * kBK * 2;
    static constexpr uint32_t kStages = kStageBudget / (kABytes + kBBytes);
    static constexpr uint32_t kSmem = kStages * (kABytes + kBBytes) + 1024;
    static constexpr uint32_t kTmemCols = 2 * BN;        // two accumulators
};

struct GemmParams {
    wr_gemm_args a;
    wr_weight w;
    uint32_t m_tiles, n_tiles, k_blocks;
    long long wait_limit;
    int *err;
};

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ uint32_t pack_bf16(float a, float b)
{
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t *>(&h);
}
__device__ __forceinline__ uint32_t pack_f16(float a, float b)
{
    const __half2 h = __floats2half2_rn(fminf(fmaxf(a, -65504.f), 65504.f), fminf(fmaxf(b, -65504.f), 65504.f));
    return *reinterpret_cast<const uint32_t *>(&h);
}

template <uint32_t BN>
__global__ void __launch_bounds__(kThreads, 1)
gemm_bf16_kernel(const __grid_constant__ CUtensorMap x_map, const GemmParams p)
{
    using T = Tile<BN>;
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t full[T::kStages], empty[T::kStages], acc_full[2], acc_empty[2];
    __shared__ uint32_t tmem_slot;
    uint8_t *stages = reinterpret_cast<uint8_t *>(((uintptr_t)smem_raw + 1023u) & ~(uintptr_t)1023u);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    if (threadIdx.x == 0) {
        for (uint32_t i = 0; i < T::kStages; ++i) {
            mbar_init(&full[i], 1);
            mbar_init(&empty[i], 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(&acc_full[i], 1);
            mbar_init(&acc_empty[i], 4);
        }
        fence_barrier_init();
    }
    if (warp == 1) tc5::alloc(&tmem_slot, T::kTmemCols);
    tc5::fence_before();
    __syncthreads();
    tc5::fence_after();
    const uint32_t tmem = tmem_slot;
    pdl_wait();
    const uint32_t m_tiles = p.a.group.list ? *p.a.group.count : p.m_tiles, tiles = m_tiles * p.n_tiles;

    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x) {
                const uint32_t m0 = (tile % m_tiles) * kBM, n0 = (tile / m_tiles) * BN;
                const char *blocks = static_cast<const char *>(p.w.blocks);
                if (p.a.group.list) blocks += p.a.group.list[tile % m_tiles] * p.a.group.stride;
                for (uint32_t kb = 0; kb < p.k_blocks; ++kb, ++it) {
                    const uint32_t st = it % T::kStages;
                    if (it >= T::kStages && !mbar_wait(&empty[st], (it / T::kStages - 1) & 1, p.wait_limit)) {
                        ok = false;
                        break;
                    }
                    uint8_t *a = stages + st * (kABytes + T::kBBytes), *b = a + kABytes;
                    const uint32_t nb0 = n0 / kWBlock, nb = min(BN / kWBlock, wr_weight_blocks(p.w.n) - nb0);
                    if (p.a.pages) {
                        const uint32_t np = m0 + kPageTokens < p.a.m ? 2u : 1u;
                        mbar_expect_tx(&full[st], np * kABytes / 2 + nb * kWBlockBytes);
                        for (uint32_t i = 0; i < np; ++i)
                            bulk_g2s(a + i * kABytes / 2, reinterpret_cast<const char *>(p.a.pages[m0 / kPageTokens + i]) + kb * kABytes / 2,
                                     kABytes / 2, &full[st]);
                    } else {
                        mbar_expect_tx(&full[st], kABytes + nb * kWBlockBytes);
                        tc5::tma_load_2d(a, &x_map, (int)(kb * kBK), (int)m0, &full[st]);
                    }
                    const char *w = blocks + ((size_t)nb0 * p.k_blocks + kb) * kWBlockBytes;
                    for (uint32_t i = 0; i < nb; ++i)
                        bulk_g2s(b + i * kWBlockBytes, w + (size_t)i * p.k_blocks * kWBlockBytes, kWBlockBytes, &full[st]);
                }
            }
            if (!ok) atomicCAS(p.err, 0, 41);
            // nothing of this CTA's may be in flight when it leaves: the last loads have landed and (unless
            // a wait ran out) the products that read them have completed
            const uint32_t last = it < T::kStages ? it : T::kStages;
            for (uint32_t i = it - last; i < it; ++i)
                (void)mbar_wait(ok ? &empty[i % T::kStages] : &full[i % T::kStages], (i / T::kStages) & 1, p.wait_limit);
        }
    } else if (warp == 1) {
        const bool lead = tc5::elect_one();
        const uint32_t idesc = p.a.pages ? tc5::idesc_f16(kBM, BN) : tc5::idesc_bf16(kBM, BN);
        uint32_t it = 0, n_tile = 0;
        bool ok = true;
        for (uint32_t tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, ++n_tile) {
            const uint32_t acc = n_tile & 1;
            if (n_tile >= 2 && !mbar_wait(&acc_empty[acc], (n_tile / 2 - 1) & 1, p.wait_limit)) {
                ok = false;
                break;
            }
            tc5::fence_after();
            for (uint32_t kb = 0; kb < p.k_blocks; ++kb, ++it) {
                const uint32_t st = it % T::kStages;
                if (!mbar_wait(&full[st], (it / T::kStages) & 1, p.wait_limit)) {
                    ok = false;
                    break;
                }
                tc5::fence_after();
                const uint32_t a_addr = smem_u32(stages + st * (kABytes + T::kBBytes));
                const uint64_t a = tc5::desc_kmajor(a_addr), b = tc5::desc_kmajor(a_addr + kABytes);
#pragma unroll
                for (uint32_t kk = 0; kk < kBK / 16; ++kk)
                    if (lead) tc5::mma_ss(tmem + acc * BN, a + 2 * kk, b + 2 * kk, idesc, (kb | kk) != 0);
                if (lead) tc5::commit(&empty[st]);
            }
            if (ok && lead) tc5::commit(&acc_full[acc]);
        }
        if (!ok && lane == 0) atomicCAS(p.err, 0, 42);
    } else {
        const uint32_t quarter = warp & 3;                       // TMEM lanes this warp may read
        uint32_t n_tile = 0;
        bool ok = true;
        for (uint32_t tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, ++n_tile) {
            const uint32_t m0 = (tile % m_tiles) * kBM, n0 = (tile / m_tiles) * BN;
            const uint32_t acc = n_tile & 1, row = m0 + quarter * 32 + lane;
            if (!mbar_wait(&acc_full[acc], (n_tile / 2) & 1, p.wait_limit)) {
                ok = false;
                break;
            }
            tc5::fence_after();
            const uint32_t n_pad = (p.w.n + 7u) & ~7u;
#pragma unroll 1
            for (uint32_t c0 = 0; c0 < BN && n0 + c0 < n_pad; c0 += 32) {
                float v[32];
                tc5::ld32(tmem + ((quarter * 32) << 16) + acc * BN + c0, v);
                tc5::wait_ld();
                if (row < p.a.m) {
#pragma unroll
                    for (uint32_t g = 0; g < 4; ++g) {
                        const uint32_t col = n0 + c0 + 8 * g;
                        if (col >= p.a.pair.from) {
                            if ((g & 1u) || col >= n_pad) continue;
                            float y[8];
#pragma unroll
                            for (int e = 0; e < 8; ++e)
                                y[e] = wr_pair_act(p.a.pair.act, p.a.pair.alpha, p.a.pair.limit, v[8 * g + e],
                                                   v[8 * ((g + 1) & 3u) + e]);
                            *reinterpret_cast<uint4 *>((__nv_bfloat16 *)p.a.pair.out + (size_t)row * p.a.pair.ld +
                                                       (col - p.a.pair.from) / 2) =
                                make_uint4(pack_bf16(y[0], y[1]), pack_bf16(y[2], y[3]), pack_bf16(y[4], y[5]),
                                           pack_bf16(y[6], y[7]));
                        } else if (col < n_pad) {
                            float *u = v + 8 * g;
                            if (p.a.bias) {
                                const float4 b0 = *reinterpret_cast<const float4 *>(p.a.bias + col);
                                const float4 b1 = *reinterpret_cast<const float4 *>(p.a.bias + col + 4);
                                u[0] += b0.x; u[1] += b0.y; u[2] += b0.z; u[3] += b0.w;
                                u[4] += b1.x; u[5] += b1.y; u[6] += b1.z; u[7] += b1.w;
                            }
                            if (p.a.act == WR_GEMM_ACT_SOFTPLUS) {
#pragma unroll
                                for (int e = 0; e < 8; ++e) u[e] = softplus(u[e]);
                            }
                            if (p.a.out_bf16)
                                *reinterpret_cast<uint4 *>((__nv_bfloat16 *)p.a.out_bf16 + (size_t)row * p.a.out_bf16_ld + col) =
                                    make_uint4(pack_bf16(u[0], u[1]), pack_bf16(u[2], u[3]), pack_bf16(u[4], u[5]),
                                               pack_bf16(u[6], u[7]));
                            if (p.a.mul != 1.f) {
#pragma unroll
                                for (int e = 0; e < 8; ++e) u[e] *= p.a.mul;
                            }
                            if (p.a.add) {
                                const float *r = p.a.add + (size_t)row * p.a.add_ld + col;
                                const float4 r0 = *reinterpret_cast<const float4 *>(r);
                                const float4 r1 = *reinterpret_cast<const float4 *>(r + 4);
                                u[0] += r0.x; u[1] += r0.y; u[2] += r0.z; u[3] += r0.w;
                                u[4] += r1.x; u[5] += r1.y; u[6] += r1.z; u[7] += r1.w;
                            }
                            const size_t at = (size_t)row * p.a.out_ld + col;
                            if (p.a.out_type == WR_GEMM_OUT_F32) {
                                float4 *o = reinterpret_cast<float4 *>((float *)p.a.out + at);
                                o[0] = make_float4(u[0], u[1], u[2], u[3]);
                                o[1] = make_float4(u[4], u[5], u[6], u[7]);
                            } else if (p.a.out_type == WR_GEMM_OUT_BF16) {
                                *reinterpret_cast<uint4 *>((__nv_bfloat16 *)p.a.out + at) =
                                    make_uint4(pack_bf16(u[0], u[1]), pack_bf16(u[2], u[3]), pack_bf16(u[4], u[5]),
                                               pack_bf16(u[6], u[7]));
                            } else {
                                *reinterpret_cast<uint4 *>((__half *)p.a.out + at) =
                                    make_uint4(pack_f16(u[0], u[1]), pack_f16(u[2], u[3]), pack_f16(u[4], u[5]),
                                               pack_f16(u[6], u[7]));
                            }
                        }
                    }
                }
            }
            tc5::fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[acc]);
        }
        if (!ok && lane == 0) atomicCAS(p.err, 0, 43);
    }
    tc5::fence_before();
    __syncthreads();
    tc5::fence_after();
    if (warp == 1) tc5::dealloc(tmem, T::kTmemCols);
}

typedef CUresult (*encode_tiled_fn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *,
                                    const cuuint64_t *, const cuuint32_t *, const cuuint32_t *,
                                    CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion,
                                    CUtensorMapFloatOOBfill);

int map_2d(CUtensorMap *map, const void *base, uint32_t rows, uint32_t k, uint32_t ld, uint32_t box_rows)
{
    static encode_tiled_fn fn = nullptr;
    if (!fn) {
        void *sym = nullptr;
        cudaDriverEntryPointQueryResult qres;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &qres) != cudaSuccess ||
            qres != cudaDriverEntryPointSuccess) {
            (void)cudaGetLastError();
            return WR_CUDA_ERR_INTERNAL;
        }
        fn = (encode_tiled_fn)sym;
    }
    const cuuint64_t dims[2] = {k, rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {kBK, box_rows};
    const cuuint32_t estr[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, estr,
              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS
               ? WR_CUDA_OK
               : WR_CUDA_ERR_INTERNAL;
}

template <uint32_t BN>
int launch(wr_cuda_ctx *ctx, const CUtensorMap &x, const wr_weight &w, const wr_gemm_args &a)
{
    constexpr uint32_t flag = BN == 256 ? 16u : BN == 128 ? 32u : 64u;
    if (!(ctx->attr_flags & flag)) {
        WR_CUDA_TRY(cudaFuncSetAttribute(gemm_bf16_kernel<BN>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)Tile<BN>::kSmem));
        ctx->attr_flags |= flag;
    }
    GemmParams p;
    p.a = a;
    p.w = w;
    p.m_tiles = (a.m + kBM - 1) / kBM;
    p.n_tiles = (w.n + BN - 1) / BN;
    p.k_blocks = wr_weight_blocks(w.k);
    p.wait_limit = ctx->wait_limit;
    p.err = ctx->dev_err;
    const uint32_t grid = std::min<uint32_t>((a.group.list ? a.group.max : p.m_tiles) * p.n_tiles, (uint32_t)ctx->sm_count);
    WR_CUDA_TRY(wr_launch_pdl(gemm_bf16_kernel<BN>, dim3(grid), dim3(kThreads), Tile<BN>::kSmem, ctx->stream, x, p));
    ctx->launches++;
    WR_CUDA_TRY(cudaGetLastError());
    return WR_CUDA_OK;
}

}  // namespace

int wr_gemm_map_rows(CUtensorMap *map, const void *x, uint32_t rows, uint32_t k, uint32_t ld)
{
    return map_2d(map, x, rows, k, ld, kBM);
}

int wr_skinny_map_rows(CUtensorMap *map, const void *split_rows, uint32_t k, uint32_t ld, uint32_t groups)
{
    return map_2d(map, split_rows, groups * 2 * WR_CUDA_BATCH_MAX, k, ld, 2 * WR_CUDA_BATCH_MAX);
}

int wr_gemm_launch(wr_cuda_ctx *ctx, const CUtensorMap &x, const wr_weight &w, const wr_gemm_args &a)
{
    if (a.m == 0 || w.n == 0 || w.k == 0 || (a.out_ld & 7u) || (a.out_bf16_ld & 7u) || (a.add_ld & 7u) ||
        (a.pair.from != ~0u && ((a.pair.from & 15u) || (a.pair.ld & 7u))))
        return WR_CUDA_ERR_INVAL;
    // the tile width that finishes first: rounds over the device times the width's share of the work
    const uint32_t m_tiles = a.group.list ? a.group.max : (a.m + kBM - 1) / kBM;
    uint32_t best = 0;
    uint64_t best_cost = ~0ull;
    for (uint32_t bn : {256u, 128u, 64u}) {
        const uint64_t tiles = (uint64_t)m_tiles * ((w.n + bn - 1) / bn);
        const uint64_t cost = ((tiles + ctx->sm_count - 1) / ctx->sm_count) * (bn + 48u);
        if (cost < best_cost) {
            best_cost = cost;
            best = bn;
        }
    }
    if (best == 256) return launch<256>(ctx, x, w, a);
    if (best == 128) return launch<128>(ctx, x, w, a);
    return launch<64>(ctx, x, w, a);
}
