// attn_latent.cu — attention of a few rows over the cached latents on the tensor cores (decode steps, short portions).
//
// All heads of a layer read the same cached row, once as key and (its first part) once as value, so a page is fetched
// once for up to 16 heads and serves both products.  Operands are swapped: keys are the tensor core's M.
//
// A work item is one row, one group of NH heads and one chunk of keys.  CTAs are persistent (one per SM at most): the next
// item's pages are on their way while this one's last tile is being worked off.  Per tile of 128 keys (two pages):
//   * warp 0 brings the pages' blocks of 64 keys x 64 values in with linear bulk copies (they are stored in the
//     operand's layout): the latent in units of 128 values, which stay until the second product has read them, the
//     rotated part in a ring of its own, free again after the first;
//   * warp 1 issues S^T[128 keys x 2 NH] = rows . queries^T and O^T[latent x 2 NH] += rows^T . P^T, the second with the
//     rows as a transposed operand.  Queries and weights are F32 split in two F16 numbers, one column each, so the
//     products see about 22 bits of them;
//   * warps 2-5, a thread per key: column maxima across the tile, exponentials, P^T to shared memory.  O^T stays in
//     TMEM and is rescaled only when a maximum has grown by more than 2^8.
// The queries come as that operand already (wr_latent_query_launch).  A chunk leaves (maximum, sum) and O in F32; the
// value kernel, or latent_merge_kernel where there are many, adds the chunks up in order.  How a session is cut into
// chunks depends on its own length alone.  Every wait is bounded by the context's wait limit.
#include <algorithm>

#include "latent_dev.cuh"
#include "tcgen05_dev.cuh"
#include "warp_reduce.cuh"

namespace {

constexpr uint32_t kTile = 128, kThreads = 192, kBox = kTile * 128, kUnit = 2 * kBox, kBlock = 8192;
constexpr uint32_t kMaxUnits = 16, kMaxRot = 8;
constexpr uint32_t kSmemMax = 232448;
constexpr float kLn2 = 0.6931471805599453f;
constexpr float kGrow = 8.0f;

// tiles per chunk, by the session's length
__host__ __device__ inline uint32_t chunk_tiles(uint32_t len)
{
    const uint32_t tiles = (len + kTile - 1) / kTile, c = (tiles + 63) / 64;
    return tiles > 16 && c < 2 ? 2u : c;
}
__host__ __device__ inline uint32_t chunk_count(uint32_t len)
{
    const uint32_t per = chunk_tiles(len) * kTile;
    return (len + per - 1) / per;
}

struct LatentParams {
    wr_rows rw;
    uint32_t heads, layer;
    uint32_t units, rot_boxes, boxes;            // per tile: pairs of latent boxes, rotated boxes; boxes of a query
    uint32_t ring, rot_ring, tmem_cols;
    uint32_t chunks;                             // of the longest row: the stride of ml and o
    uint32_t items, groups;                      // work items; groups of heads
    wr_latent_lens lens;
    const char *q;                               // [rows][head groups][boxes][2 NH][128 B]
    size_t q_row;
    float *ml, *o;                               // [rows][heads][chunks][2], [rows][heads][chunks][rank_pad]
    uint32_t rank_pad;
    long long wait_limit;
    int *err;
};

struct LatentBars {
    uint64_t full[kMaxUnits], empty[kMaxUnits], rot_full[kMaxRot], rot_empty[kMaxRot];
    uint64_t q_full, q_empty, s_full, p_full, o_full, o_free;
    uint32_t tmem;
    alignas(16) float red[2][16][4];             // per head: the four warps' maxima (or sums)
};

template <int M> __device__ __forceinline__ uint32_t warp_max_many(float (&v)[M], uint32_t lane)
{
    uint32_t width = M, idx = 0;
#pragma unroll
    for (uint32_t o = 16; o >= 1; o >>= 1) {
        if (width > 1) {
            const uint32_t half = width / 2;
            const bool upper = (lane & o) != 0;
#pragma unroll
            for (uint32_t i = 0; i < M / 2; ++i)
                if (i < half) {
                    const float send = upper ? v[i] : v[i + half], keep = upper ? v[i + half] : v[i];
                    v[i] = fmaxf(keep, __shfl_xor_sync(0xffffffffu, send, o));
                }
            if (upper) idx += half;
            width = half;
        } else {
            v[0] = fmaxf(v[0], __shfl_xor_sync(0xffffffffu, v[0], o));
        }
    }
    return idx;
}
__device__ __forceinline__ void group_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ float ex2(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
struct Item {
    uint32_t row, group, chunk, len, tile0, tiles;
};
__device__ __forceinline__ Item item_of(const LatentParams &p, uint32_t i)
{
    Item it;
    it.group = i % p.groups;
    i /= p.groups;
    it.row = 0;
    while (i >= p.lens.count[it.row]) i -= p.lens.count[it.row++];
    it.chunk = i;
    it.len = p.lens.len[it.row];
    const uint32_t per = chunk_tiles(it.len);
    it.tile0 = i * per;
    it.tiles = min(per, (it.len + kTile - 1) / kTile - it.tile0);
    return it;
}

template <int NH>
__global__ void __launch_bounds__(kThreads, 1) latent_decode_kernel(const LatentParams p)
{
    constexpr uint32_t N = 2 * NH;
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t *const units = smem_raw, *const rots = units + p.ring * kUnit, *const qs = rots + p.rot_ring * kBox;
    uint8_t *const ps = qs + p.boxes * N * 128;          // [2 key boxes][N][128 B]
    LatentBars &sm = *reinterpret_cast<LatentBars *>(ps + 2 * N * 128);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    if (threadIdx.x == 0) {
        for (uint32_t i = 0; i < p.ring; ++i) {
            mbar_init(&sm.full[i], 1);
            mbar_init(&sm.empty[i], 1);
        }
        for (uint32_t i = 0; i < p.rot_ring; ++i) {
            mbar_init(&sm.rot_full[i], 1);
            mbar_init(&sm.rot_empty[i], 1);
        }
        mbar_init(&sm.q_full, 1);
        mbar_init(&sm.q_empty, 1);
        mbar_init(&sm.s_full, 1);
        mbar_init(&sm.p_full, 4);
        mbar_init(&sm.o_full, 1);
        mbar_init(&sm.o_free, 4);
        fence_barrier_init();
    }
    if (warp == 1) tc5::alloc(&sm.tmem, p.tmem_cols);
    tc5::fence_before();
    __syncthreads();
    tc5::fence_after();
    pdl_wait();
    const uint32_t tmem_s = sm.tmem, tmem_o = tmem_s + 32;       // (S: 32 columns whatever N is)

    if (warp == 0) {
        if (lane == 0) {                                 // the pages
            const uint32_t rank_boxes = p.boxes - p.rot_boxes;
            uint32_t n_unit = 0, n_rot = 0;              // requested so far
            bool ok = true;
            for (uint32_t i = blockIdx.x; i < p.items && ok; i += gridDim.x) {
                const Item it = item_of(p, i);
                const wr_seq_dev s = p.rw.seqs[seq_of(p.rw, it.row)];
                const uint64_t *table = s.pages + (size_t)p.layer * s.n_pages;
                const uint32_t last_page = (it.len - 1) / kPageTokens;
                for (uint32_t t = 0; t < it.tiles && ok; ++t) {
                    // (a tile's second page may lie behind the last one: the first comes twice, its weights are zeros)
                    const uint32_t pg = (it.tile0 + t) * 2;
                    const char *src[2] = {reinterpret_cast<const char *>(table[pg]),
                                          reinterpret_cast<const char *>(table[min(pg + 1, last_page)])};
                    for (uint32_t u = 0; u < p.units && ok; ++u, ++n_unit) {
                        const uint32_t st = n_unit % p.ring;
                        if (n_unit >= p.ring && !mbar_wait(&sm.empty[st], (n_unit / p.ring - 1) & 1, p.wait_limit)) {
                            ok = false;
                            break;
                        }
                        const uint32_t nb = min(2u, rank_boxes - 2 * u);
                        mbar_expect_tx(&sm.full[st], nb * kBox);
                        for (uint32_t b = 0; b < nb; ++b)
                            for (uint32_t h = 0; h < 2; ++h)
                                bulk_g2s(units + st * kUnit + b * kBox + h * kBlock, src[h] + (2 * u + b) * kBlock, kBlock,
                                         &sm.full[st]);
                    }
                    for (uint32_t r = 0; r < p.rot_boxes && ok; ++r, ++n_rot) {
                        const uint32_t st = n_rot % p.rot_ring;
                        if (n_rot >= p.rot_ring && !mbar_wait(&sm.rot_empty[st], (n_rot / p.rot_ring - 1) & 1, p.wait_limit)) {
                            ok = false;
                            break;
                        }
                        mbar_expect_tx(&sm.rot_full[st], kBox);
                        for (uint32_t h = 0; h < 2; ++h)
                            bulk_g2s(rots + st * kBox + h * kBlock, src[h] + (rank_boxes + r) * kBlock, kBlock, &sm.rot_full[st]);
                    }
                }
            }
            if (!ok) atomicCAS(p.err, 0, 61);
            // nothing in flight when the CTA leaves
            for (uint32_t i = n_unit - min(n_unit, p.ring); i < n_unit; ++i)
                (void)mbar_wait(&sm.full[i % p.ring], (i / p.ring) & 1, p.wait_limit);
            for (uint32_t i = n_rot - min(n_rot, p.rot_ring); i < n_rot; ++i)
                (void)mbar_wait(&sm.rot_full[i % p.rot_ring], (i / p.rot_ring) & 1, p.wait_limit);
        } else if (lane == 1) {                          // the queries
            uint32_t n = 0;
            bool ok = true;
            for (uint32_t i = blockIdx.x; i < p.items; i += gridDim.x, ++n) {
                if (n > 0) ok = mbar_wait(&sm.q_empty, (n - 1) & 1, p.wait_limit);
                if (!ok) break;
                const Item it = item_of(p, i);
                mbar_expect_tx(&sm.q_full, p.boxes * N * 128);
                bulk_g2s(qs, p.q + it.row * p.q_row + (size_t)it.group * p.boxes * N * 128, p.boxes * N * 128, &sm.q_full);
            }
            if (!ok) atomicCAS(p.err, 0, 64);
            if (n > 0) (void)mbar_wait(&sm.q_full, (n - 1) & 1, p.wait_limit);
        }
        __syncwarp();
    } else if (warp == 1) {
        const bool lead = tc5::elect_one();
        constexpr uint32_t idesc_s = tc5::idesc_f16(kTile, N), idesc_o = idesc_s | tc5::kIdescAMnMajor;
        const uint32_t q_addr = smem_u32(qs), p_addr = smem_u32(ps);
        uint32_t n_unit = 0, n_rot = 0, n_tile = 0, n_item = 0;
        bool ok = true;
        for (uint32_t i = blockIdx.x; i < p.items && ok; i += gridDim.x, ++n_item) {
            const Item it = item_of(p, i);
            ok = mbar_wait(&sm.q_full, n_item & 1, p.wait_limit);
            if (!ok) break;
            for (uint32_t t = 0; t < it.tiles && ok; ++t, ++n_tile) {
                // S^T, box by box as they arrive
                uint32_t box = 0;
                auto score = [&](uint32_t rows) {
                    const uint64_t a = tc5::desc_kmajor(rows), b = tc5::desc_kmajor(q_addr + box * N * 128);
#pragma unroll
                    for (uint32_t kk = 0; kk < 4; ++kk)
                        if (lead) tc5::mma_ss(tmem_s, a + 2 * kk, b + 2 * kk, idesc_s, (box | kk) != 0);
                    ++box;
                };
                for (uint32_t u = 0; u < p.units && ok; ++u) {
                    const uint32_t j = n_unit + u, st = j % p.ring;
                    ok = mbar_wait(&sm.full[st], (j / p.ring) & 1, p.wait_limit);
                    if (!ok) break;
                    tc5::fence_after();
                    score(smem_u32(units + st * kUnit));
                    if (2 * u + 1 < p.boxes - p.rot_boxes) score(smem_u32(units + st * kUnit + kBox));
                }
                for (uint32_t r = 0; r < p.rot_boxes && ok; ++r, ++n_rot) {
                    const uint32_t st = n_rot % p.rot_ring;
                    ok = mbar_wait(&sm.rot_full[st], (n_rot / p.rot_ring) & 1, p.wait_limit);
                    if (!ok) break;
                    tc5::fence_after();
                    score(smem_u32(rots + st * kBox));
                    if (lead) tc5::commit(&sm.rot_empty[st]);
                }
                if (!ok) break;
                if (lead) {
                    if (t + 1 == it.tiles) tc5::commit(&sm.q_empty);
                    tc5::commit(&sm.s_full);
                }
                ok = mbar_wait(&sm.p_full, n_tile & 1, p.wait_limit);
                // the item's first product overwrites O: the one before must have left TMEM
                if (ok && t == 0 && n_item > 0) ok = mbar_wait(&sm.o_free, (n_item - 1) & 1, p.wait_limit);
                if (!ok) break;
                tc5::fence_after();
                // O^T: 128 latents of a unit at a time, 16 keys a step
                for (uint32_t u = 0; u < p.units; ++u, ++n_unit) {
                    const uint32_t st = n_unit % p.ring;
                    const uint64_t a = tc5::desc_mnmajor(smem_u32(units + st * kUnit), kBox), b = tc5::desc_kmajor(p_addr);
#pragma unroll
                    for (uint32_t kk = 0; kk < kTile / 16; ++kk)
                        if (lead)
                            tc5::mma_ss(tmem_o + u * N, a + kk * (2048 >> 4), b + (kk >> 2) * (N * 128 >> 4) + (kk & 3) * 2,
                                        idesc_o, (t | kk) != 0);
                    if (lead) tc5::commit(&sm.empty[st]);
                }
            }
            if (ok && lead) tc5::commit(&sm.o_full);
        }
        if (!ok && lane == 0) atomicCAS(p.err, 0, 62);
        __syncwarp();
    } else {
        const uint32_t quarter = warp & 3, key = quarter * 32 + lane, tid = threadIdx.x - 64, lanes = (quarter * 32) << 16;
        uint32_t n_tile = 0, n_item = 0, n_red = 0;
        bool ok = true;
        // (a warp whose wait ran out goes through the motions: the group's barriers count on all four)
        for (uint32_t i = blockIdx.x; i < p.items; i += gridDim.x, ++n_item) {
            const Item it = item_of(p, i);
            const uint32_t head0 = it.group * NH, nh = min((uint32_t)NH, p.heads - head0);
            float m[NH], l[NH];
#pragma unroll
            for (int h = 0; h < NH; ++h) {
                m[h] = WR_NEG_SENTINEL;
                l[h] = 0.f;
            }
            for (uint32_t t = 0; t < it.tiles; ++t, ++n_tile, ++n_red) {
                if (ok) ok = mbar_wait(&sm.s_full, n_tile & 1, p.wait_limit);    // (the tile before has been multiplied: P is quiet)
                ok = __all_sync(0xffffffffu, ok);
                tc5::fence_after();
                float v[32];
                tc5::ld32(tmem_s + lanes, v);
                tc5::wait_ld();
                const bool seen = (it.tile0 + t) * kTile + key < it.len;
                float sc[NH], mx[NH];
#pragma unroll
                for (int h = 0; h < NH; ++h) mx[h] = sc[h] = seen ? v[h] + v[NH + h] : WR_NEG_SENTINEL;
                const uint32_t idx = warp_max_many<NH>(mx, lane), b = n_red & 1;
                sm.red[b][idx][quarter] = mx[0];                 // (lanes that share an index hold one value)
                group_sync();
                bool grow = false;
                float a[NH];
#pragma unroll
                for (int h = 0; h < NH; ++h) {
                    const float4 w = *reinterpret_cast<const float4 *>(sm.red[b][h]);
                    const float top = fmaxf(fmaxf(w.x, w.y), fmaxf(w.z, w.w));
                    a[h] = 1.0f;
                    if (t == 0) {
                        m[h] = top;
                    } else if (top > m[h] + kGrow) {
                        a[h] = ex2(m[h] - top);
                        m[h] = top;
                        grow = true;
                    }
                }
                if (grow) {                                      // (the same in all threads)
#pragma unroll
                    for (int h = 0; h < NH; ++h) l[h] *= a[h];
#pragma unroll 1
                    for (uint32_t c = 0; c < p.units * N; c += 32) {
                        tc5::ld32(tmem_o + lanes + c, v);
                        tc5::wait_ld();
#pragma unroll
                        for (int e = 0; e < 32; ++e) v[e] *= a[e % NH];
                        tc5::st32(tmem_o + lanes + c, v);
                    }
                    tc5::wait_st();
                }
#pragma unroll
                for (int h = 0; h < NH; ++h) {
                    const float w = ex2(sc[h] - m[h]);
                    l[h] += w;
                    const __half hi = __float2half_rn(w);
                    *reinterpret_cast<__half *>(ps + wr_latent_split_off(N, h, key)) = hi;
                    *reinterpret_cast<__half *>(ps + wr_latent_split_off(N, NH + h, key)) = __float2half_rn(w - __half2float(hi));
                }
                fence_proxy_async();
                tc5::fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(&sm.p_full);
            }
            if (ok) ok = mbar_wait(&sm.o_full, n_item & 1, p.wait_limit);
            ok = __all_sync(0xffffffffu, ok);
            tc5::fence_after();
            const size_t at = ((size_t)it.row * p.heads + head0) * p.chunks + it.chunk, stride = (size_t)p.chunks * p.rank_pad;
            float *out = p.o + at * p.rank_pad;
#pragma unroll 1
            for (uint32_t c = 0; c < p.units * N; c += 32) {
                float v[32];
                tc5::ld32(tmem_o + lanes + c, v);
                tc5::wait_ld();
#pragma unroll
                for (uint32_t j = 0; j < 32 / N; ++j) {
                    const uint32_t d = (c / N + j) * 128 + key;
#pragma unroll
                    for (uint32_t h = 0; h < NH; ++h)
                        if (h < nh && d < p.rank_pad) out[h * stride + d] = v[j * N + h] + v[j * N + NH + h];
                }
            }
            tc5::fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&sm.o_free);
            // the sums: across the warp's keys, then the four warps in order
            const uint32_t idx = warp_reduce_many<NH>(l, lane), b = n_red++ & 1;
            sm.red[b][idx][quarter] = l[0];
            group_sync();
#pragma unroll
            for (uint32_t h = 0; h < NH; ++h)
                if (tid == h && h < nh) {
                    const float4 w = *reinterpret_cast<const float4 *>(sm.red[b][h]);
                    *reinterpret_cast<float2 *>(p.ml + 2 * (at + (size_t)h * p.chunks)) =
                        make_float2(m[h] * kLn2, ((w.x + w.y) + w.z) + w.w);
                }
        }
        if (!ok && lane == 0) atomicCAS(p.err, 0, 63);
    }
    tc5::fence_before();
    __syncthreads();
    tc5::fence_after();
    if (warp == 1) tc5::dealloc(sm.tmem, p.tmem_cols);
}

// Chunks of a row and head added up, in order.
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentParams p, float *out)
{
    __shared__ float w[64];
    pdl_trigger();
    pdl_wait();
    const uint32_t head = blockIdx.x, row = blockIdx.y, n = p.lens.count[row];
    const size_t at = ((size_t)row * p.heads + head) * p.chunks;
    if (threadIdx.x < 32) latent_chunk_weights(p.ml + 2 * at, n, w, threadIdx.x);
    __syncthreads();
    for (uint32_t c = 4 * threadIdx.x; c < p.rank_pad; c += 512)
        store4(out + ((size_t)row * p.heads + head) * p.rank_pad + c, latent_chunk_sum(p.o + at * p.rank_pad + c, p.rank_pad, w, n));
}

// sizes of the rings; 0: it does not fit
uint32_t plan(const wr_latent_geom &g, uint32_t nh, LatentParams &p)
{
    const uint32_t n = 2 * nh, rank_boxes = g.rank_pad() / 64;
    p.boxes = g.row() / 64;
    p.rot_boxes = p.boxes - rank_boxes;
    p.units = (rank_boxes + 1) / 2;
    const uint32_t fixed = p.boxes * n * 128 + 2 * n * 128 + (uint32_t)sizeof(LatentBars);
    p.rot_ring = p.rot_boxes;
    p.ring = 0;
    while (p.ring < kMaxUnits && fixed + (p.ring + 1) * kUnit + p.rot_ring * kBox <= kSmemMax) ++p.ring;
    if (p.ring < p.units || p.rot_ring > kMaxRot) return 0;
    while (p.rot_ring + p.rot_boxes <= kMaxRot && p.rot_ring < 3 * p.rot_boxes && p.ring > 2 * p.units) {
        p.rot_ring += p.rot_boxes;                       // tiles far enough ahead: as many of their rotated parts
        while (fixed + p.ring * kUnit + p.rot_ring * kBox > kSmemMax) --p.ring;
    }
    p.tmem_cols = 32;
    while (p.tmem_cols < 32 + (p.units * n + 31) / 32 * 32) p.tmem_cols *= 2;
    return fixed + p.ring * kUnit + p.rot_ring * kBox;
}

template <int NH> int launch(wr_cuda_ctx *ctx, const LatentParams &p, uint32_t smem)
{
    WR_CUDA_TRY(cudaFuncSetAttribute(latent_decode_kernel<NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    WR_CUDA_TRY(wr_launch_pdl(latent_decode_kernel<NH>, dim3(std::min<uint32_t>(p.items, ctx->sm_count)), dim3(kThreads),
                              (size_t)smem, ctx->stream, p));
    return finish_launch(ctx);
}

}  // namespace

bool wr_latent_decode_covers(const wr_latent_geom &g)
{
    LatentParams p{};
    return g.dim_pad() <= 512 && plan(g, wr_latent_group(g), p) != 0;
}

int wr_latent_decode_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_latent_geom &g, uint32_t layer, const void *q,
                            const uint32_t *lens, float *merged, wr_latent_value_args &out)
{
    LatentParams p{};
    const uint32_t nh = wr_latent_group(g), smem = plan(g, nh, p);
    if (!smem || rw.n_rows > WR_CUDA_BATCH_MAX) return WR_CUDA_ERR_LIMIT;
    p.rw = rw;
    p.heads = g.heads;
    p.rank_pad = g.rank_pad();
    p.layer = layer;
    for (uint32_t r = 0; r < rw.n_rows; ++r) {
        p.lens.len[r] = lens[r];
        p.lens.count[r] = chunk_count(lens[r]);
        p.chunks = std::max(p.chunks, p.lens.count[r]);
        p.items += p.lens.count[r];
    }
    p.groups = (g.heads + nh - 1) / nh;
    p.items *= p.groups;
    const size_t pieces = (size_t)rw.n_rows * g.heads * p.chunks, ml = (pieces * 2 + 63) & ~(size_t)63;
    int rc = wr_ctx_reserve_ws(ctx, (ml + pieces * p.rank_pad) * sizeof(float), 0);
    if (rc != WR_CUDA_OK) return rc;
    p.q = static_cast<const char *>(q);
    p.q_row = wr_latent_split_bytes(g);
    p.ml = ctx->ws;
    p.o = ctx->ws + ml;
    p.wait_limit = ctx->wait_limit;
    p.err = ctx->dev_err;
    rc = nh == 8 ? launch<8>(ctx, p, smem) : launch<16>(ctx, p, smem);
    if (rc != WR_CUDA_OK) return rc;
    out.lens = p.lens;
    out.chunks = p.chunks;
    out.ml = p.ml;
    out.o = p.o;
    // (few enough: every block of the value kernel adds them up for itself; the same sums either way)
    if (p.chunks <= kLatentMaxFused && rw.n_rows * p.chunks <= 32) return WR_CUDA_OK;
    WR_CUDA_TRY(wr_launch_pdl(latent_merge_kernel, dim3(g.heads, rw.n_rows), dim3(128), 0, ctx->stream, p, merged));
    out.ml = nullptr;
    out.o = merged;
    return finish_launch(ctx);
}
