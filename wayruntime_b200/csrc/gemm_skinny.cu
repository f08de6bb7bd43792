// gemm_skinny.cu — out[r][n] = act(w[n] . x[r] + bias) + add for up to 16 rows: a decode step's projections.
//
// HBM-bound: the weights are all the traffic.  The operands are swapped — 128 weight rows are the tensor core's M,
// the activation rows its N, each F32 activation as two BF16 numbers in two columns (split rows, see
// gemm_bf16.cuh).  A CTA owns 128 weight rows and a slice of K; the CTAs of a cluster share the rows and add their
// slices up, in rank order, out of each other's shared memory.  Warp 0 streams both operands with TMA — the weights
// depend on nothing, so their first stages are requested before the kernel ahead has finished —, warp 1 issues
// tcgen05.mma, warps 2-5 finish the rows.  All columns are always computed: a row's result does not depend on how
// many rows share the step.
#include <cuda_bf16.h>

#include <algorithm>

#include "gemm_bf16.cuh"
#include "tcgen05_dev.cuh"

namespace {

constexpr uint32_t kRows = WR_CUDA_BATCH_MAX, kM = 128, kN = 2 * kRows, kBK = 64;
constexpr uint32_t kThreads = 192, kStages = 5;
constexpr uint32_t kABytes = kM * kBK * 2, kBBytes = kN * kBK * 2, kStageBytes = kABytes + kBBytes;
constexpr uint32_t kMaxSplit = 8;
constexpr uint32_t kTmemCols = 32;
static_assert(kRows * kM * 4 <= kStages * kStageBytes, "a CTA's sums fit where its stages were");

struct SkinnyParams {
    wr_skinny_args a;
    wr_weight w;
    uint32_t k_blocks, split;
    long long wait_limit;
    int *err;
};

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ float load_rank(const float *p, uint32_t rank)
{
    uint32_t remote;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(smem_u32(p)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
    return v;
}

// row i as split rows: the value's rounding, and what is left kRows rows behind it
__device__ __forceinline__ void put_split(void *out, uint32_t ld, uint32_t i, uint32_t n, float y)
{
    __nv_bfloat16 *o = static_cast<__nv_bfloat16 *>(out) + (size_t)i * ld + n;
    const __nv_bfloat16 hi = __float2bfloat16_rn(y);
    o[0] = hi;
    o[(size_t)kRows * ld] = __float2bfloat16_rn(y - __bfloat162float(hi));
}

// a gate row and the up row that belongs to it
__device__ __forceinline__ void put_pair(const SkinnyParams &p, uint32_t group, uint32_t i, uint32_t n, float g, float u)
{
    if (n >= p.w.n) return;
    const uint32_t c = n - p.a.pair.from;
    put_split(p.a.pair.out, p.a.pair.ld, 2 * kRows * group + i, c / 16 * 8 + (c & 7u),
              wr_pair_act(p.a.pair.act, p.a.pair.alpha, p.a.pair.limit, g, u));
}

// bias, activation, copies and residual of one finished sum: activation row i, weight row n
__device__ __forceinline__ void put(const SkinnyParams &p, uint32_t group, uint32_t i, uint32_t n, float y)
{
    if (n >= p.w.n) return;
    if (p.a.bias) y += p.a.bias[n];
    if (p.a.act == WR_GEMM_ACT_SOFTPLUS) y = softplus(y);
    if (p.a.out_split) put_split(p.a.out_split, p.a.out_split_ld, i, n, y);
    y *= p.a.mul;
    if (p.a.add) y += p.a.add[(size_t)i * p.a.add_ld + n];
    p.a.out[((size_t)kRows * group + i) * p.a.out_ld + n] = y;
}

__global__ void __launch_bounds__(kThreads)
gemm_skinny_kernel(const __grid_constant__ CUtensorMap x_map, const SkinnyParams p)
{
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t full[kStages], empty[kStages], acc_full;
    __shared__ uint32_t tmem_slot;
    uint8_t *stages = reinterpret_cast<uint8_t *>(((uintptr_t)smem_raw + 1023u) & ~(uintptr_t)1023u);
    float *red = reinterpret_cast<float *>(stages);      // [row][128], once the products are done
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t rank = blockIdx.x % p.split, n0 = (blockIdx.x / p.split) * kM;
    const uint32_t kb0 = p.k_blocks * rank / p.split, kb1 = p.k_blocks * (rank + 1) / p.split, nkb = kb1 - kb0;
    const uint32_t group = blockIdx.y;
    const char *blocks = static_cast<const char *>(p.w.blocks);
    pdl_trigger();
    if (p.a.group.list) {                                // (the same answer in every CTA of a cluster)
        pdl_wait();
        if (group >= *p.a.group.count) return;
        blocks += p.a.group.list[group] * p.a.group.stride;
    }
    if (threadIdx.x == 0) {
        for (uint32_t i = 0; i < kStages; ++i) {
            mbar_init(&full[i], 1);
            mbar_init(&empty[i], 1);
        }
        mbar_init(&acc_full, 1);
        fence_barrier_init();
    }
    if (warp == 1) tc5::alloc(&tmem_slot, kTmemCols);
    tc5::fence_before();
    __syncthreads();
    tc5::fence_after();
    const uint32_t tmem = tmem_slot;
    float s[kRows];

    if (warp == 0) {
        if (lane == 0) {
            asm volatile("prefetch.tensormap [%0];" ::"l"(&x_map) : "memory");
            // the row tile's one or two blocks of weights
            const uint32_t nb = min(kM / kWBlock, wr_weight_blocks(p.w.n) - n0 / kWBlock);
            const char *w = blocks + ((size_t)(n0 / kWBlock) * p.k_blocks + kb0) * kWBlockBytes;
            const uint64_t policy = l2_policy_evict_first();         // streamed once
            auto weights = [&](uint32_t it) {
                const uint32_t st = it % kStages;
                uint8_t *a = stages + st * kStageBytes;
                mbar_expect_tx(&full[st], nb * kWBlockBytes + kBBytes);
                for (uint32_t i = 0; i < nb; ++i)
                    bulk_g2s_hint(a + i * kWBlockBytes, w + ((size_t)i * p.k_blocks + it) * kWBlockBytes, kWBlockBytes, &full[st],
                                  policy);
            };
            auto rows = [&](uint32_t it) {
                const uint32_t st = it % kStages;
                tc5::tma_load_2d(stages + st * kStageBytes + kABytes, &x_map, (int)((kb0 + it) * kBK), (int)(p.a.group.x_rows * group),
                                 &full[st]);
            };
            bool ok = true;
            uint32_t it = 0;
            const uint32_t first = nkb < kStages ? nkb : kStages;
            for (; it < first; ++it) weights(it);
            pdl_wait();
            for (uint32_t i = 0; i < first; ++i) rows(i);
            for (; it < nkb; ++it) {
                if (!mbar_wait(&empty[it % kStages], (it / kStages - 1) & 1, p.wait_limit)) {
                    ok = false;
                    break;
                }
                weights(it);
                rows(it);
            }
            if (!ok) atomicCAS(p.err, 0, 51);
            const uint32_t last = it < kStages ? it : kStages;
            for (uint32_t i = it - last; i < it; ++i)    // nothing in flight when the CTA leaves
                (void)mbar_wait(ok ? &empty[i % kStages] : &full[i % kStages], (i / kStages) & 1, p.wait_limit);
        }
        __syncwarp();
    } else if (warp == 1) {
        const bool lead = tc5::elect_one();
        constexpr uint32_t idesc = tc5::idesc_bf16(kM, kN);
        bool ok = true;
        for (uint32_t it = 0; it < nkb; ++it) {
            const uint32_t st = it % kStages;
            if (!mbar_wait(&full[st], (it / kStages) & 1, p.wait_limit)) {
                ok = false;
                break;
            }
            tc5::fence_after();
            const uint32_t addr = smem_u32(stages + st * kStageBytes);
            const uint64_t a = tc5::desc_kmajor(addr), b = tc5::desc_kmajor(addr + kABytes);
#pragma unroll
            for (uint32_t kk = 0; kk < kBK / 16; ++kk)
                if (lead) tc5::mma_ss(tmem, a + 2 * kk, b + 2 * kk, idesc, (it | kk) != 0);
            if (lead) tc5::commit(&empty[st]);
        }
        if (ok && lead) tc5::commit(&acc_full);
        if (!ok && lane == 0) atomicCAS(p.err, 0, 52);
        __syncwarp();
    } else {
        pdl_wait();
        if (!mbar_wait(&acc_full, 0, p.wait_limit) && lane == 0) atomicCAS(p.err, 0, 53);
        __syncwarp();
        tc5::fence_after();
        float v[kN];
        tc5::ld32(tmem + (((warp & 3) * 32) << 16), v);  // lane: weight row; column: activation row
        tc5::wait_ld();
#pragma unroll
        for (uint32_t i = 0; i < kRows; ++i) s[i] = v[i] + v[kRows + i];
    }
    const uint32_t m = (warp & 3) * 32 + lane;           // (finishing warps)
    if (p.split == 1) {
        if (warp >= 2) {
#pragma unroll
            for (uint32_t i = 0; i < kRows; ++i)
                if (i < p.a.rows) {
                    const float up = __shfl_xor_sync(0xffffffffu, s[i], 8);
                    if (n0 + m < p.a.pair.from) put(p, group, i, n0 + m, s[i]);
                    else if (!(m & 8u)) put_pair(p, group, i, n0 + m, s[i], up);
                }
        }
    } else {
        // every rank lays its sums out in its own shared memory (its products are done with it) and finishes its
        // share of the weight rows from all of them
        if (warp >= 2) {
#pragma unroll
            for (uint32_t i = 0; i < kRows; ++i)
                if (i < p.a.rows) red[i * kM + m] = s[i];
        }
        cluster_arrive();
        cluster_wait();
        if (warp >= 2) {
            const uint32_t share = kM / p.split;
            for (uint32_t j = threadIdx.x - 64; j < p.a.rows * share; j += kThreads - 64) {
                const uint32_t i = j / share, mm = rank * share + j % share;
                auto sum = [&](uint32_t at) {
                    float v[kMaxSplit];
#pragma unroll
                    for (uint32_t q = 0; q < kMaxSplit; ++q) v[q] = q < p.split ? load_rank(red + i * kM + at, q) : 0.f;
                    float y = v[0];
#pragma unroll
                    for (uint32_t q = 1; q < kMaxSplit; ++q) y += v[q];  // (+0 beyond the last rank)
                    return y;
                };
                if (n0 + mm < p.a.pair.from) put(p, group, i, n0 + mm, sum(mm));
                else if (!(mm & 8u)) put_pair(p, group, i, n0 + mm, sum(mm), sum(mm + 8));
            }
        }
        cluster_arrive();                                // nobody leaves while its sums are being read
        cluster_wait();
    }
    tc5::fence_before();
    __syncthreads();
    tc5::fence_after();
    if (warp == 1) tc5::dealloc(tmem, kTmemCols);
}

}  // namespace

int wr_skinny_launch(wr_cuda_ctx *ctx, const CUtensorMap &x, const wr_weight &w, const wr_skinny_args &a)
{
    if (a.rows == 0 || a.rows > kRows || w.n == 0 || w.k == 0) return WR_CUDA_ERR_INVAL;
    SkinnyParams p;
    p.a = a;
    p.w = w;
    p.k_blocks = wr_weight_blocks(w.k);
    p.wait_limit = ctx->wait_limit;
    p.err = ctx->dev_err;
    if (a.pair.from != ~0u && (a.pair.from & 15u)) return WR_CUDA_ERR_INVAL;
    const uint32_t tiles = (w.n + kM - 1) / kM, groups = a.group.list ? a.group.max : 1u;
    // two CTAs per SM where a slice still has a few blocks of K (with groups: `usual` of them at a time; the split has
    // to be the same whatever the step holds)
    const uint32_t usual = tiles * (a.group.list ? a.group.usual : 1u), room = (a.group.list ? 1.3 : 2.0) * ctx->sm_count;
    p.split = 1;
    while (p.split < kMaxSplit && usual * p.split * 2 <= room && p.k_blocks >= 8 * p.split) p.split *= 2;
    constexpr size_t smem = kStages * kStageBytes + 1024;
    if (!(ctx->attr_flags & 128u)) {
        WR_CUDA_TRY(cudaFuncSetAttribute(gemm_skinny_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        ctx->attr_flags |= 128u;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(tiles * p.split, groups);
    cfg.blockDim = dim3(kThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = p.split;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = p.split > 1 ? 2 : 1;
    WR_CUDA_TRY(cudaLaunchKernelEx(&cfg, gemm_skinny_kernel, x, p));
    ctx->launches++;
    WR_CUDA_TRY(cudaGetLastError());
    return WR_CUDA_OK;
}
