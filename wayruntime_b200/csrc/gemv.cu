// gemv.cu — y[r][n] = sum_k W[n][k] x[r][k] in F32 for a few activation rows: weights stream from HBM once.
//
// Serves every projection of the F32 layer stack (src/core/kernels.c:978-1090: GGML-layout W[out][in]) and those
// of the mixed stack's F32 models.
#include <math.h>

#include "gemv.cuh"
#include "warp_reduce.cuh"

namespace {

constexpr int kGemvThreads = 128;      // 4 warps per CTA
constexpr int kGemvWarps = kGemvThreads / 32;
constexpr int kChunk = 512;            // activation floats staged per row and pass

__device__ __forceinline__ float4 ldg_stream(const float *p)
{
    float4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.f32 {%0,%1,%2,%3}, [%4];"
                 : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w)
                 : "l"(p));
    return v;
}

// ---- the GEMV pair ---------------------------------------------------------
//
// y[r][n] = sum_k W[n][k] * x[r][k], optionally with RMSNorm fused on x, and a
// residual add or SiLU(gate)*up on the way out.  Two kernels, one arithmetic:
// K is cut into four quarters; inside a quarter lane l takes the 16-byte
// vectors l, l+32, ... in ascending order with fused multiply-adds, starting
// from zero; lane l then adds its four quarter sums in order; the 32 lane sums
// are added by the xor butterfly (offsets 16, 8, 4, 2, 1).  The fused norm
// multiplies x by the norm weight first and the finished sum by
// 1/sqrt(mean(x^2)+eps) last, the sum of squares following the same quarter /
// lane / butterfly order.  Because both kernels compute every output by exactly
// this recipe, a row's bits do not depend on how many rows share the call or on
// which kernel served it.
//
//   gemv_splitk_kernel (<= 4 activation rows): a CTA owns C weight rows and
//     its four warps take one quarter each, so every lane has all its loads in
//     flight at once and nothing is staged; x comes straight from L2.  With few
//     rows the weights are all the traffic, and one warp per weight row would
//     leave most of the device idle on a narrow output (1024 rows = 7 warps/SM).
//   gemv_rows_kernel (up to 16 rows per CTA): each warp owns NW weight rows
//     and walks the four quarters itself; the activation rows of the current
//     piece of a quarter sit in shared memory for all four warps, so x costs
//     RG/(4*NW) of the weight bytes instead of RG/C.

struct KQuarters {
    uint32_t vec, per;     // 16-byte vectors in K; vectors per quarter
    __device__ __forceinline__ explicit KQuarters(uint32_t k) : vec(k / 4), per((k / 4 + 3) / 4) {}
    __device__ __forceinline__ uint32_t lo(uint32_t q) const { return q * per < vec ? q * per : vec; }
    __device__ __forceinline__ uint32_t hi(uint32_t q) const { return (q + 1) * per < vec ? (q + 1) * per : vec; }
};

__device__ __forceinline__ float sumsq4(float ss, const float4 v)
{
    return fmaf(v.w, v.w, fmaf(v.z, v.z, fmaf(v.y, v.y, fmaf(v.x, v.x, ss))));
}
__device__ __forceinline__ float4 mul4(const float4 a, const float4 b)
{
    return make_float4(__fmul_rn(a.x, b.x), __fmul_rn(a.y, b.y), __fmul_rn(a.z, b.z), __fmul_rn(a.w, b.w));
}
__device__ __forceinline__ float dot4(const float4 w, const float4 x, float acc)
{
    acc = fmaf(w.x, x.x, acc);
    acc = fmaf(w.y, x.y, acc);
    acc = fmaf(w.z, x.z, acc);
    return fmaf(w.w, x.w, acc);
}
__device__ __forceinline__ float inv_rms_of(float sumsq, uint32_t k, float eps)
{
    return 1.0f / sqrtf(__fadd_rn(__fdiv_rn(sumsq, (float)k), eps));
}
__device__ __forceinline__ float silu_mul(float g, float u)
{
    return __fmul_rn(__fdiv_rn(g, __fadd_rn(1.0f, expf(-g))), u);
}

__device__ __forceinline__ float softplus(float x)
{
    return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x)));
}
// bias and activation of a finished sum, then the residual
__device__ __forceinline__ float finish(const GemvParams &p, uint32_t s, uint32_t n, uint32_t row, float y)
{
    if (p.bias && s == 0) y = __fadd_rn(y, p.bias[n]);
    if (p.act == WR_GEMV_ACT_SOFTPLUS) y = softplus(y);
    y = __fmul_rn(y, p.mul);
    if (p.add) y = __fadd_rn(p.add[(size_t)row * p.add_stride + n], y);
    return y;
}

// weight rows of a CTA / warp: plain, or swiglu (first half gate rows, second half the same rows of up)
template <int NR>
__device__ __forceinline__ void weight_rows(const GemvParams &p, const GemvSeg &seg, uint32_t n0,
                                            const float *(&wrow)[NR])
{
    constexpr int H = (NR >= 2) ? NR / 2 : 1;
#pragma unroll
    for (int c = 0; c < NR; ++c) {
        uint32_t n = p.swiglu ? n0 + (c % H) : n0 + c;
        const float *base = p.swiglu ? ((c < H) ? p.seg[0].w : p.seg[1].w) : seg.w;
        if (n >= seg.n) n = seg.n - 1;               // clamped rows are computed and dropped
        wrow[c] = base + (size_t)n * p.k;
    }
}

constexpr int kPrefetchRegs = 16;        // 16-byte weight vectors a lane holds before the dependency wait

template <int RG, int C>
__global__ void __launch_bounds__(kGemvThreads) gemv_splitk_kernel(const GemvParams p)
{
    __shared__ float part[kGemvWarps][C * RG + RG][32];      // per quarter (= warp): every lane's partial sums
    __shared__ float red[C * RG + RG];
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t r0 = blockIdx.y * RG;
    uint32_t cta = blockIdx.x, s = 0;
    if (!p.swiglu) {
        while (s + 1 < p.n_seg && cta >= p.cta_end[s]) ++s;
        if (s > 0) cta -= p.cta_end[s - 1];
    }
    const GemvSeg seg = p.seg[s];
    constexpr int H = (C >= 2) ? C / 2 : 1;
    const uint32_t n0 = cta * (p.swiglu ? H : C);
    const float *wrow[C];
    weight_rows<C>(p, seg, n0, wrow);
    const float *xrow[RG];
#pragma unroll
    for (int r = 0; r < RG; ++r) {
        const uint32_t row = (r0 + r < p.rows) ? r0 + r : p.rows - 1;    // clamped rows are dropped at the end
        xrow[r] = p.x + (size_t)row * p.x_stride;
    }
    const KQuarters kq(p.k);
    const uint32_t v_lo = kq.lo(warp), v_hi = kq.hi(warp);

    float acc[C][RG], ss[RG];
#pragma unroll
    for (int r = 0; r < RG; ++r) {
        ss[r] = 0.f;
#pragma unroll
        for (int c = 0; c < C; ++c) acc[c][r] = 0.f;
    }
    // Weights do not depend on the kernel before this one: the first PV vectors of the lane's walk
    // (all of it for K up to 512 * PV) are requested before the dependency wait, so their trip from
    // HBM overlaps that kernel's tail; the activations are read after it.
    constexpr int PV = kPrefetchRegs / C;
    float4 wbuf[PV][C];
#pragma unroll
    for (int i = 0; i < PV; ++i) {
        const uint32_t v = v_lo + lane + 32u * i;
        if (v < v_hi) {
#pragma unroll
            for (int c = 0; c < C; ++c) wbuf[i][c] = ldg_stream(wrow[c] + 4 * v);
        }
    }
    pdl_wait();
    auto step = [&](uint32_t v, const float4 (&w)[C]) {
        float4 nw = make_float4(1.f, 1.f, 1.f, 1.f);
        if (p.norm_w) nw = *reinterpret_cast<const float4 *>(p.norm_w + 4 * v);
#pragma unroll
        for (int r = 0; r < RG; ++r) {
            float4 xv = *reinterpret_cast<const float4 *>(xrow[r] + 4 * v);
            if (p.norm_w) {
                ss[r] = sumsq4(ss[r], xv);
                xv = mul4(xv, nw);
            }
#pragma unroll
            for (int c = 0; c < C; ++c) acc[c][r] = dot4(w[c], xv, acc[c][r]);
        }
    };
#pragma unroll
    for (int i = 0; i < PV; ++i) {
        const uint32_t v = v_lo + lane + 32u * i;
        if (v < v_hi) step(v, wbuf[i]);
    }
#pragma unroll 2
    for (uint32_t v = v_lo + lane + 32u * PV; v < v_hi; v += 32) {
        float4 w[C];
#pragma unroll
        for (int c = 0; c < C; ++c) w[c] = ldg_stream(wrow[c] + 4 * v);
        step(v, w);
    }
    constexpr int M = C * RG;
#pragma unroll
    for (int i = 0; i < M; ++i) part[warp][i][lane] = acc[i / RG][i % RG];
    if (p.norm_w) {
#pragma unroll
        for (int r = 0; r < RG; ++r) part[warp][M + r][lane] = ss[r];
    }
    __syncthreads();
    // every lane adds its four quarter sums in order, then the butterfly over the lanes
    for (int idx = warp; idx < M + (p.norm_w ? RG : 0); idx += kGemvWarps) {
        float t = part[0][idx][lane];
#pragma unroll
        for (int q = 1; q < kGemvWarps; ++q) t = __fadd_rn(t, part[q][idx][lane]);
#pragma unroll
        for (int o = 16; o >= 1; o >>= 1) t = __fadd_rn(t, __shfl_xor_sync(0xffffffffu, t, o));
        if (lane == 0) red[idx] = t;
    }
    __syncthreads();
    const int n_out = p.swiglu ? H * RG : C * RG;
    if (tid < n_out) {
        const int c = tid / RG, r = tid % RG;
        const uint32_t n = n0 + c, row = r0 + r;
        if (n < seg.n && row < p.rows) {
            const float inv = p.norm_w ? inv_rms_of(red[M + r], p.k, p.eps) : 1.0f;
            float y = __fmul_rn(red[c * RG + r], inv);
            if (p.swiglu) {
                const float u = __fmul_rn(red[(c + H) * RG + r], inv);
                seg.out[(size_t)row * seg.out_stride + n] = silu_mul(y, u);
            } else {
                seg.out[(size_t)row * seg.out_stride + n] = finish(p, s, n, row, y);
            }
        }
    }
}

// RG: activation rows per CTA (row group); NW: weight rows per warp.
template <int RG, int NW>
__global__ void __launch_bounds__(kGemvThreads) gemv_rows_kernel(const GemvParams p)
{
    constexpr int kPieceVec = kChunk / 4;            // 16-byte vectors of x staged per row and pass
    __shared__ __align__(16) float xs[RG][kChunk];
    __shared__ float inv_rms[RG];
    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t r0 = blockIdx.y * RG;
    uint32_t cta = blockIdx.x, s = 0;
    if (!p.swiglu) {
        while (s + 1 < p.n_seg && cta >= p.cta_end[s]) ++s;
        if (s > 0) cta -= p.cta_end[s - 1];
    }
    const GemvSeg seg = p.seg[s];
    constexpr int H = (NW >= 2) ? NW / 2 : 1;
    const uint32_t n0 = (cta * kGemvWarps + warp) * (p.swiglu ? H : NW);
    const float *wrow[NW];
    weight_rows<NW>(p, seg, n0, wrow);
    const KQuarters kq(p.k);
    pdl_wait();

    if (p.norm_w) {                                  // sum of squares in the shared order
        for (int r = warp; r < RG; r += kGemvWarps) {
            float t = 0.f;
            if (r0 + r < p.rows) {
                const float *xr = p.x + (size_t)(r0 + r) * p.x_stride;
#pragma unroll 1
                for (uint32_t q = 0; q < 4; ++q) {
                    float ss = 0.f;
                    for (uint32_t v = kq.lo(q) + lane; v < kq.hi(q); v += 32)
                        ss = sumsq4(ss, *reinterpret_cast<const float4 *>(xr + 4 * v));
                    t = (q == 0) ? ss : __fadd_rn(t, ss);
                }
            }
#pragma unroll
            for (int o = 16; o >= 1; o >>= 1) t = __fadd_rn(t, __shfl_xor_sync(0xffffffffu, t, o));
            if (lane == 0) inv_rms[r] = inv_rms_of(t, p.k, p.eps);
        }
    }

    constexpr int M = NW * RG;
    constexpr int G = (M > 32) ? 32 : M;
    constexpr int NG = M / G;
    float lane_tot[NW][RG];                          // this lane's quarter sums, added in quarter order

#pragma unroll 1
    for (uint32_t q = 0; q < 4; ++q) {
        const uint32_t v_lo = kq.lo(q), v_hi = kq.hi(q);
        float acc[NW][RG];
#pragma unroll
        for (int c = 0; c < NW; ++c)
#pragma unroll
            for (int r = 0; r < RG; ++r) acc[c][r] = 0.f;
        for (uint32_t c0 = v_lo; c0 < v_hi; c0 += kPieceVec) {
            const uint32_t nvec = (v_hi - c0 < (uint32_t)kPieceVec) ? v_hi - c0 : (uint32_t)kPieceVec;
            __syncthreads();                         // the previous piece has been consumed
            for (uint32_t i = tid; i < RG * nvec; i += kGemvThreads) {
                const uint32_t r = i / nvec, vv = i % nvec;
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (r0 + r < p.rows) {
                    v = *reinterpret_cast<const float4 *>(p.x + (size_t)(r0 + r) * p.x_stride + 4 * (c0 + vv));
                    if (p.norm_w) v = mul4(v, *reinterpret_cast<const float4 *>(p.norm_w + 4 * (c0 + vv)));
                }
                *reinterpret_cast<float4 *>(&xs[r][4 * vv]) = v;
            }
            __syncthreads();
#pragma unroll 2
            for (uint32_t vv = lane; vv < nvec; vv += 32) {
                float4 w[NW];
#pragma unroll
                for (int c = 0; c < NW; ++c) w[c] = ldg_stream(wrow[c] + 4 * (c0 + vv));
#pragma unroll
                for (int r = 0; r < RG; ++r) {
                    const float4 xv = *reinterpret_cast<const float4 *>(&xs[r][4 * vv]);
#pragma unroll
                    for (int c = 0; c < NW; ++c) acc[c][r] = dot4(w[c], xv, acc[c][r]);
                }
            }
        }
#pragma unroll
        for (int c = 0; c < NW; ++c)
#pragma unroll
            for (int r = 0; r < RG; ++r) lane_tot[c][r] = (q == 0) ? acc[c][r] : __fadd_rn(lane_tot[c][r], acc[c][r]);
    }
    // the butterfly over the lanes, once, for all NW * RG sums
    float tot[NG];
    int tot_idx[NG];
#pragma unroll
    for (int g = 0; g < NG; ++g) {
        float v[G];
#pragma unroll
        for (int i = 0; i < G; ++i) v[i] = lane_tot[(g * G + i) / RG][(g * G + i) % RG];
        tot_idx[g] = warp_reduce_many<G>(v, lane) + g * G;
        tot[g] = v[0];
    }
    __syncthreads();                                 // inv_rms is complete (and visible) for every warp

    if (!p.swiglu) {
#pragma unroll
        for (int g = 0; g < NG; ++g) {
            const uint32_t c = tot_idx[g] / RG, r = tot_idx[g] % RG, n = n0 + c, row = r0 + r;
            if (reduce_writer<G>(lane) && n < seg.n && row < p.rows) {
                float y = __fmul_rn(tot[g], p.norm_w ? inv_rms[r] : 1.0f);
                seg.out[(size_t)row * seg.out_stride + n] = finish(p, s, n, row, y);
            }
        }
    } else if constexpr (NW >= 2) {
        // flat index = c * RG + r over all NW rows: gate rows are c < H, up rows c >= H.  A lane that
        // holds gate (c, r) needs up (c + H, r): with M <= 32 it sits in the same group at index
        // + H*RG, whose owner differs in one lane bit; with two groups it is this lane's other total.
        if constexpr (NG == 2) {
            const uint32_t c = tot_idx[0] / RG, r = tot_idx[0] % RG, n = n0 + c, row = r0 + r;
            // group 0 holds rows [0, 32/RG) = gate, group 1 the same positions of up
            if (n < seg.n && row < p.rows) {
                const float inv = p.norm_w ? inv_rms[r] : 1.0f;
                seg.out[(size_t)row * seg.out_stride + n] =
                    silu_mul(__fmul_rn(tot[0], inv), __fmul_rn(tot[1], inv));
            }
        } else {
            // index bits are the top log2(M) lane bits; + H*RG = + M/2 flips the highest one (lane bit 4)
            const float other = __shfl_xor_sync(0xffffffffu, tot[0], 16);
            const uint32_t c = tot_idx[0] / RG, r = tot_idx[0] % RG, n = n0 + c, row = r0 + r;
            if (reduce_writer<G>(lane) && c < (uint32_t)H && n < seg.n && row < p.rows) {
                const float inv = p.norm_w ? inv_rms[r] : 1.0f;
                seg.out[(size_t)row * seg.out_stride + n] =
                    silu_mul(__fmul_rn(tot[0], inv), __fmul_rn(other, inv));
            }
        }
    }
}

template <int RG, int NW>
void launch_gemv_t(const GemvParams &p, uint32_t ctas, cudaStream_t st)
{
    dim3 grid(ctas, (p.rows + RG - 1) / RG);
    (void)wr_launch_pdl(gemv_rows_kernel<RG, NW>, grid, dim3(kGemvThreads), 0, st, p);
}

template <int RG, int C>
void launch_splitk_t(const GemvParams &p, uint32_t ctas, cudaStream_t st)
{
    dim3 grid(ctas, (p.rows + RG - 1) / RG);
    (void)wr_launch_pdl(gemv_splitk_kernel<RG, C>, grid, dim3(kGemvThreads), 0, st, p);
}

template <int C>
void launch_splitk(const GemvParams &p, uint32_t ctas, cudaStream_t st)
{
    if (p.rows == 1) launch_splitk_t<1, C>(p, ctas, st);
    else if (p.rows == 2) launch_splitk_t<2, C>(p, ctas, st);
    else launch_splitk_t<4, C>(p, ctas, st);
}

template <int NW>
void launch_gemv_rg(const GemvParams &p, uint32_t ctas, cudaStream_t st)
{
    const uint32_t r = p.rows;
    if (r == 1) launch_gemv_t<1, NW>(p, ctas, st);
    else if (r == 2) launch_gemv_t<2, NW>(p, ctas, st);
    else if (r <= 4) launch_gemv_t<4, NW>(p, ctas, st);
    else if (r <= 8) launch_gemv_t<8, NW>(p, ctas, st);
    else launch_gemv_t<16, NW>(p, ctas, st);
}

// Weight rows per warp from the total output width: narrow outputs take one row
// per warp so that the grid still covers the device.
int weight_rows_per_warp(uint32_t n_total)
{
    if (n_total >= 32768) return 4;
    if (n_total >= 2048) return 2;
    return 1;
}


constexpr uint32_t kSplitKRowsMax = 4;

}  // namespace

int wr_gemv_launch(wr_cuda_ctx *ctx, GemvParams &p, uint32_t n_total_for_width)
{
    if (p.rows <= kSplitKRowsMax) {
        // weight rows per CTA: 2 for narrow outputs (more CTAs), 4 otherwise
        const int c = (p.swiglu || n_total_for_width >= 4096) ? 4 : 2;
        const uint32_t cols_per_cta = p.swiglu ? (uint32_t)c / 2 : (uint32_t)c;
        uint32_t ctas = 0;
        if (p.swiglu) {
            ctas = (p.seg[0].n + cols_per_cta - 1) / cols_per_cta;
        } else {
            for (uint32_t s = 0; s < p.n_seg; ++s) {
                ctas += (p.seg[s].n + cols_per_cta - 1) / cols_per_cta;
                p.cta_end[s] = ctas;
            }
        }
        if (c == 4) launch_splitk<4>(p, ctas, ctx->stream);
        else launch_splitk<2>(p, ctas, ctx->stream);
        WR_CUDA_TRY(cudaGetLastError());
        return WR_CUDA_OK;
    }
    const int nw = p.swiglu ? 2 : weight_rows_per_warp(n_total_for_width);
    const uint32_t cols_per_cta = (p.swiglu ? 1u : (uint32_t)nw) * kGemvWarps;
    uint32_t ctas = 0;
    if (p.swiglu) {
        ctas = (p.seg[0].n + cols_per_cta - 1) / cols_per_cta;
    } else {
        for (uint32_t s = 0; s < p.n_seg; ++s) {
            ctas += (p.seg[s].n + cols_per_cta - 1) / cols_per_cta;
            p.cta_end[s] = ctas;
        }
    }
    cudaStream_t st = ctx->stream;
    if (nw == 4) launch_gemv_rg<4>(p, ctas, st);
    else if (nw == 2) launch_gemv_rg<2>(p, ctas, st);
    else launch_gemv_rg<1>(p, ctas, st);
    WR_CUDA_TRY(cudaGetLastError());
    return WR_CUDA_OK;
}
