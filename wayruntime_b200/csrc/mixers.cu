// mixers.cu — row kernels of the mixed layer stack (model_mixed.cu): embedding with positions, grouped RMS
// norm with token shift, PolyNorm, causal convolution, selective scan, and what surrounds attention.
//
// All arithmetic is F32; activation rows that only feed a BF16 matrix product are stored in its type.  Rows are
// wr_ld(n) values apart; the pad columns are written as zeros, so that a weight-streaming product may read whole
// 16-byte vectors.  A row's result depends on its session alone: the same code serves a prompt's portion and a
// decode step, whatever else is in the step.
#include <cuda_bf16.h>

#include <algorithm>
#include <type_traits>

#include "rows_dev.cuh"

namespace {

// ------------------------------------------------------------------ embedding

template <typename TW>
__global__ void __launch_bounds__(256) embed_kernel(const wr_rows rw, const uint32_t *tokens, const TW *table,
                                                    const double *turns, float *x, uint32_t width, float scale)
{
    pdl_trigger();
    pdl_wait();
    const uint32_t row = blockIdx.y, ld = wr_ld(width);
    const uint32_t pos = rw.seqs[seq_of(rw, row)].pos + tok_of(rw, row);
    const TW *src = table + (size_t)tokens[row] * ld;
    float *dst = x + (size_t)row * ld;
    // a pair of columns shares its angle; ld is even
    for (uint32_t i = 2 * (blockIdx.x * 256 + threadIdx.x); i < ld; i += 2 * gridDim.x * 256) {
        float v0 = i < width ? to_f32(src[i]) * scale : 0.f, v1 = i + 1 < width ? to_f32(src[i + 1]) * scale : 0.f;
        if (turns && i < width) {
            // the angle in turns, reduced before it leaves double: a position of 2^20 keeps its phase
            const double a = turns[i >> 1] * (double)pos;
            float sn, cs;
            sincospif(2.0f * (float)(a - rint(a)), &sn, &cs);
            v0 += sn;
            if (i + 1 < width) v1 += cs;
        }
        *reinterpret_cast<float2 *>(dst + i) = make_float2(v0, v1);
    }
}

// ------------------------------------------------------- grouped norm, token shift

constexpr uint32_t kNormThreads = 256, kNormWarps = kNormThreads / 32;

// 1 / root mean square of every group of a row -> inv[groups], of its deviations from the group's mean -> mean[groups]
// with `centre` (mean: zeros without); part: groups * split partial sums
__device__ __forceinline__ void group_inv_rms(const float *x, uint32_t groups, uint32_t gs, uint32_t split, float eps,
                                              bool centre, float *part, float *mean, float *inv)
{
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t per = (gs + split - 1) / split;
    if (centre) {
        for (uint32_t u = warp; u < groups * split; u += kNormWarps) {
            const uint32_t g = u / split, lo = (u % split) * per, hi = min(lo + per, gs);
            const float *xg = x + (size_t)g * gs;
            float s = 0.f;
            for (uint32_t i = lo + lane; i < hi; i += 32) s += xg[i];
            s = warp_sum(s);
            if (lane == 0) part[u] = s;
        }
        __syncthreads();
    }
    for (uint32_t g = threadIdx.x; g < groups; g += kNormThreads) {
        float s = 0.f;
        for (uint32_t i = 0; centre && i < split; ++i) s += part[g * split + i];
        mean[g] = s / (float)gs;
    }
    __syncthreads();
    for (uint32_t u = warp; u < groups * split; u += kNormWarps) {
        const uint32_t g = u / split, lo = (u % split) * per, hi = min(lo + per, gs);
        const float *xg = x + (size_t)g * gs;
        float ss = 0.f;
        const float m = mean[g];
        for (uint32_t i = lo + lane; i < hi; i += 32) ss = fmaf(xg[i] - m, xg[i] - m, ss);
        ss = warp_sum(ss);
        if (lane == 0) part[u] = ss;
    }
    __syncthreads();
    for (uint32_t g = threadIdx.x; g < groups; g += kNormThreads) {
        float ss = 0.f;
        for (uint32_t s = 0; s < split; ++s) ss += part[g * split + s];
        inv[g] = 1.0f / sqrtf(ss / (float)gs + eps);
    }
    __syncthreads();
}

template <typename TO>
__global__ void __launch_bounds__(kNormThreads) group_norm_kernel(const wr_rows rw, const wr_norm_args a, uint32_t split)
{
    extern __shared__ float sm_norm[];
    float *inv = sm_norm, *inv_before = inv + a.groups, *mean = inv_before + a.groups, *mean_before = mean + a.groups,
          *part = mean_before + a.groups;
    pdl_trigger();
    pdl_wait();
    const uint32_t row = blockIdx.x, ld = wr_ld(a.width), gs = a.width / a.groups;
    const float *x = a.x + (size_t)(a.gather ? a.gather[row] : row) * ld;
    const Out<TO> out(a.out, row, ld);
    group_inv_rms(x, a.groups, gs, split, a.eps, a.centre, part, mean, inv);
    if (!a.shift) {
        for (uint32_t i = threadIdx.x; i < ld; i += kNormThreads)
            out.put(i, i < a.width ? (x[i] - mean[i / gs]) * inv[i / gs] * a.w[i] : 0.f);
        return;
    }
    // the mixer reads h + (h' - h) * shift with h' the token before: this step's previous row (its norm is
    // worked out again here), or the row the session's last step left
    const wr_seq_dev s = rw.seqs[seq_of(rw, row)];
    const uint32_t t = tok_of(rw, row);
    const float *xb = x - ld;
    if (t > 0) group_inv_rms(xb, a.groups, gs, split, a.eps, a.centre, part, mean_before, inv_before);
    const float *kept = reinterpret_cast<const float *>(s.st_in + a.state_off);
    float *keep = reinterpret_cast<float *>(s.st_out + a.state_off);
    for (uint32_t i = threadIdx.x; i < ld; i += kNormThreads) {
        float y = 0.f;
        if (i < a.width) {
            const float h = (x[i] - mean[i / gs]) * inv[i / gs] * a.w[i];
            float before = 0.f;
            if (t > 0) before = (xb[i] - mean_before[i / gs]) * inv_before[i / gs] * a.w[i];
            else if (!s.fresh) before = kept[i];
            y = h + (before - h) * a.shift[i];
            if (t + 1 == s.n) keep[i] = h;
        }
        out.put(i, y);
    }
}

// The same for rows that cut evenly into NW warps' parts of at most 128 * NV values, none across a group border:
// each warp keeps its part (and the previous row's) in registers between the sum and the scaling.
template <typename TO, int NW, int NV>
__global__ void __launch_bounds__(NW * 32) group_norm_reg_kernel(const wr_rows rw, const wr_norm_args a)
{
    __shared__ float part[4][NW];
    pdl_trigger();
    const uint32_t row = blockIdx.x, ld = wr_ld(a.width), unit = a.width / NW, per_group = NW / a.groups;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, at = warp * unit + 4 * lane;
    float4 w[NV], sh[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const bool in = 4 * lane + 128 * i < unit;
        w[i] = in ? load4(a.w + at + 128 * i) : make_float4(0, 0, 0, 0);
        if (a.shift) sh[i] = in ? load4(a.shift + at + 128 * i) : make_float4(0, 0, 0, 0);
    }
    pdl_wait();
    const float *x = a.x + (size_t)(a.gather ? a.gather[row] : row) * ld + at, *xb = x - ld;
    const Out<TO> out(a.out, row, ld);
    uint32_t t = 0, n = 0, fresh = 0;
    const float *kept = nullptr;
    float *keep = nullptr;
    if (a.shift) {
        const wr_seq_dev &s = rw.seqs[seq_of(rw, row)];
        t = tok_of(rw, row);
        n = s.n;
        fresh = s.fresh;
        kept = reinterpret_cast<const float *>(s.st_in + a.state_off) + at;
        keep = reinterpret_cast<float *>(s.st_out + a.state_off) + at;
    }
    float4 v[NV], b[NV];
    float ss = 0.f, sb = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        v[i] = b[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (4 * lane + 128 * i < unit) {
            v[i] = load4(x + 128 * i);
            if (a.shift) {
                if (t > 0) b[i] = load4(xb + 128 * i);
                else if (!fresh) b[i] = load4(kept + 128 * i);
            }
        }
    }
    const uint32_t g0 = warp / per_group * per_group;
    const float gs = (float)(a.width / a.groups);
    if (a.centre) {                                              // the group's mean comes off first (not off a kept row)
        float s = 0.f, q = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
            q += (b[i].x + b[i].y) + (b[i].z + b[i].w);
        }
        s = warp_sum(s);
        q = warp_sum(q);
        if (lane == 0) { part[2][warp] = s; part[3][warp] = q; }
        __syncthreads();
        s = q = 0.f;
        for (uint32_t i = 0; i < per_group; ++i) {
            s += part[2][g0 + i];
            q += part[3][g0 + i];
        }
        s /= gs;
        q = t > 0 ? q / gs : 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (4 * lane + 128 * i < unit) {
                v[i] = make_float4(v[i].x - s, v[i].y - s, v[i].z - s, v[i].w - s);
                b[i] = make_float4(b[i].x - q, b[i].y - q, b[i].z - q, b[i].w - q);
            }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        ss = fmaf(v[i].w, v[i].w, fmaf(v[i].z, v[i].z, fmaf(v[i].y, v[i].y, fmaf(v[i].x, v[i].x, ss))));
        sb = fmaf(b[i].w, b[i].w, fmaf(b[i].z, b[i].z, fmaf(b[i].y, b[i].y, fmaf(b[i].x, b[i].x, sb))));
    }
    ss = warp_sum(ss);
    sb = warp_sum(sb);
    if (lane == 0) { part[0][warp] = ss; part[1][warp] = sb; }
    __syncthreads();
    ss = sb = 0.f;
    for (uint32_t i = 0; i < per_group; ++i) {
        ss += part[0][g0 + i];
        sb += part[1][g0 + i];
    }
    const float inv = 1.0f / sqrtf(ss / gs + a.eps), inv_b = 1.0f / sqrtf(sb / gs + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        if (4 * lane + 128 * i >= unit) continue;
        float4 h = make_float4(v[i].x * inv * w[i].x, v[i].y * inv * w[i].y, v[i].z * inv * w[i].z, v[i].w * inv * w[i].w);
        if (a.shift) {
            float4 p = b[i];                                     // (the row a step left is kept normed)
            if (t > 0) p = make_float4(p.x * inv_b * w[i].x, p.y * inv_b * w[i].y, p.z * inv_b * w[i].z, p.w * inv_b * w[i].w);
            if (t + 1 == n) store4(keep + 128 * i, h);
            h = make_float4(h.x + (p.x - h.x) * sh[i].x, h.y + (p.y - h.y) * sh[i].y, h.z + (p.z - h.z) * sh[i].z,
                            h.w + (p.w - h.w) * sh[i].w);
        }
        out.put4(at + 128 * i, h);
    }
    if (warp == NW - 1 && lane < ld - a.width) out.put(a.width + lane, 0.f);                 // pad columns
}

template <typename TO, int NW> bool group_norm_reg(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_norm_args &a, cudaError_t &e)
{
    if (NW % a.groups || a.width % (4 * NW)) return false;
    const uint32_t vecs = (a.width / NW + 127) / 128;
    const dim3 grid(rw.n_rows), block(NW * 32);
    if (vecs <= 2) e = wr_launch_pdl(group_norm_reg_kernel<TO, NW, 2>, grid, block, 0, ctx->stream, rw, a);
    else if (vecs <= 4) e = wr_launch_pdl(group_norm_reg_kernel<TO, NW, 4>, grid, block, 0, ctx->stream, rw, a);
    else if (vecs <= 8) e = wr_launch_pdl(group_norm_reg_kernel<TO, NW, 8>, grid, block, 0, ctx->stream, rw, a);
    else return false;
    return true;
}

template <typename TO> cudaError_t norm_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_norm_args &a)
{
    // few rows: more warps on each (which kernel serves a row is a matter of the step's kind, not of its row count)
    cudaError_t e = cudaSuccess;
    if (rw.n_rows <= WR_CUDA_BATCH_MAX ? group_norm_reg<TO, 16>(ctx, rw, a, e) : group_norm_reg<TO, 8>(ctx, rw, a, e)) return e;
    const uint32_t split = std::max(1u, kNormWarps / a.groups);
    const size_t smem = (size_t)(4 * a.groups + a.groups * split) * 4;
    return wr_launch_pdl(group_norm_kernel<TO>, dim3(rw.n_rows), dim3(kNormThreads), smem, ctx->stream, rw, a, split);
}

// -------------------------------------------------------------------- PolyNorm

constexpr uint32_t kPolyThreads = 512, kPolyWarps = kPolyThreads / 32;

template <typename T, typename TO>
__global__ void __launch_bounds__(kPolyThreads) polynorm_kernel(const wr_polynorm_args a)
{
    __shared__ float red[3][kPolyWarps];
    pdl_trigger();
    pdl_wait();
    const uint32_t ld = wr_ld(a.ff), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const T *z = static_cast<const T *>(a.z) + (size_t)blockIdx.x * ld;
    const Out<TO> out(a.out, blockIdx.x, ld);
    float s1 = 0.f, s2 = 0.f, s3 = 0.f;
    for (uint32_t i = 8 * threadIdx.x; i < a.ff; i += 8 * kPolyThreads) {
        float v[8];
        load8v(z + i, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            if (i + e >= a.ff) v[e] = 0.f;
            const float v2 = v[e] * v[e], v3 = v2 * v[e];
            s1 = fmaf(v[e], v[e], s1);
            s2 = fmaf(v2, v2, s2);
            s3 = fmaf(v3, v3, s3);
        }
    }
    s1 = warp_sum(s1);
    s2 = warp_sum(s2);
    s3 = warp_sum(s3);
    if (lane == 0) { red[0][warp] = s1; red[1][warp] = s2; red[2][warp] = s3; }
    __syncthreads();
    float k[3];
#pragma unroll
    for (int p = 0; p < 3; ++p) {
        float t = 0.f;
#pragma unroll
        for (uint32_t w = 0; w < kPolyWarps; ++w) t += red[p][w];
        k[p] = 1.0f / sqrtf(t / (float)a.ff + a.eps);
    }
    const float ka = a.a * k[0], kb = a.b * k[1], kc = a.c * k[2];
    for (uint32_t i = 8 * threadIdx.x; i < ld; i += 8 * kPolyThreads) {
        float v[8];
        load8v(z + i, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = i + e < a.ff ? fmaf(v[e], fmaf(v[e], fmaf(v[e], kc, kb), ka), a.e) : 0.f;
        out.put8(i, v);
    }
}

// ----------------------------------------------------------------- convolution

constexpr uint32_t kConvThreads = 128, kConvRows = 16;

// A thread takes four channels through kConvRows tokens; with TAPS > 0 the last inputs stay in registers, with
// TAPS = 0 (any number) each is fetched again.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvThreads) conv_silu_kernel(const wr_rows rw, const wr_conv_args a)
{
    pdl_trigger();
    const uint32_t ld = wr_ld(a.inner), c = 4 * (blockIdx.x * kConvThreads + threadIdx.x), taps = TAPS ? TAPS : a.taps, tail = taps - 1;
    if (c >= ld) {
        pdl_wait();
        return;
    }
    constexpr int R = TAPS ? TAPS : 1;
    float4 w[R];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = load4(a.w + (size_t)j * ld + c);
    const float4 bias = load4(a.b + c);
    pdl_wait();
    const uint32_t seq = blockIdx.z, row0 = row0_of(rw, seq);
    const wr_seq_dev s = rw.seqs[seq];
    const T *x = static_cast<const T *>(a.x) + (size_t)row0 * a.x_ld + c;
    T *out = static_cast<T *>(a.out) + (size_t)row0 * ld + c;
    const uint32_t t0 = blockIdx.y * kConvRows, t1 = min(t0 + kConvRows, s.n);
    const float *kept = reinterpret_cast<const float *>(s.st_in + a.state_off) + c;      // [taps-1][ld]
    auto input = [&](int32_t t) -> float4 {                                              // token t of this step; < 0: before it
        if (t >= 0) return load4(x + (size_t)t * a.x_ld);
        return s.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(kept + (size_t)((int32_t)tail + t) * ld);
    };
    auto step = [](float4 &acc, const float4 wj, const float4 v) {
        acc = make_float4(fmaf(wj.x, v.x, acc.x), fmaf(wj.y, v.y, acc.y), fmaf(wj.z, v.z, acc.z), fmaf(wj.w, v.w, acc.w));
    };
    float4 win[R];
#pragma unroll
    for (int j = 1; j < TAPS; ++j) win[j] = input((int32_t)t0 + j - TAPS);
    for (uint32_t t = t0; t < t1; t += 4) {
        float4 next[4];
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int i = 0; i < 4; ++i)
                if (t + i < t1) next[i] = load4(x + (size_t)(t + i) * a.x_ld);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            if (t + i >= t1) break;
            float4 acc = bias;
            if constexpr (TAPS > 0) {
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j) win[j] = win[j + 1];
                win[TAPS - 1] = next[i];
#pragma unroll
                for (int j = 0; j < TAPS; ++j) step(acc, w[j], win[j]);
            } else {
                for (uint32_t j = 0; j < taps; ++j)
                    step(acc, load4(a.w + (size_t)j * ld + c), input((int32_t)(t + i + j) - (int32_t)tail));
            }
            acc = make_float4(siluf(acc.x), siluf(acc.y), siluf(acc.z), siluf(acc.w));
            store4(out + (size_t)(t + i) * ld, acc);
            if (a.out_split) Out<Split>(a.out_split, row0 + t + i, ld).put4(c, acc);
        }
    }
    if (t1 == s.n) {                                                                     // the block with the last token
        float *keep = reinterpret_cast<float *>(s.st_out + a.state_off) + c;
        for (uint32_t k = 0; k < tail; ++k)
            store4(keep + (size_t)k * ld, input((int32_t)(s.n + k) - (int32_t)tail));
    }
}

template <typename T> cudaError_t conv_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_conv_args &a)
{
    const uint32_t n = rw.decode ? 1u : rw.n_rows;
    const dim3 grid((wr_ld(a.inner) / 4 + kConvThreads - 1) / kConvThreads, (n + kConvRows - 1) / kConvRows, rw.n_seq), block(kConvThreads);
    if (a.taps == 4) return wr_launch_pdl(conv_silu_kernel<T, 4>, grid, block, 0, ctx->stream, rw, a);
    return wr_launch_pdl(conv_silu_kernel<T, 0>, grid, block, 0, ctx->stream, rw, a);
}

// -------------------------------------------------------------- selective scan
//
// A thread carries NS states of one channel through the step's tokens; the threads of a channel are
// neighbouring lanes and add their parts of y with shuffles.  Token tiles (x, z, dt of the block's channels, B, C)
// come in through a two-deep cp.async ring.  The state is F32 throughout.

constexpr uint32_t kScanThreads = 128;

__device__ __forceinline__ float ex2(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
template <int BYTES> __device__ __forceinline__ void cp_async(void *dst, const void *src)
{
    asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(smem_u32(dst)), "l"(src), "n"(BYTES) : "memory");
}

// The states of a thread: NS values, two to a register pair where there are two.
template <int NS> struct States {
    static constexpr int P = NS / 2;
    uint64_t v[P];
    __device__ __forceinline__ void load(const float *p)
    {
        if constexpr (NS == 2) {
            v[0] = *reinterpret_cast<const uint64_t *>(p);
        } else {
#pragma unroll
            for (int j = 0; j < P; j += 2) {
                const ulonglong2 u = *reinterpret_cast<const ulonglong2 *>(p + 2 * j);
                v[j] = u.x;
                v[j + 1] = u.y;
            }
        }
    }
    __device__ __forceinline__ void scale(float f)
    {
        const uint64_t ff = pack2(f, f);
#pragma unroll
        for (int j = 0; j < P; ++j) v[j] = mul2(v[j], ff);
    }
    // 2^(f * a)
    __device__ __forceinline__ void decay(float f, const States &a)
    {
        const uint64_t ff = pack2(f, f);
#pragma unroll
        for (int j = 0; j < P; ++j) {
            float x, y;
            unpack2(mul2(a.v[j], ff), x, y);
            v[j] = pack2(ex2(x), ex2(y));
        }
    }
    // this = e * this + b
    __device__ __forceinline__ void advance(const States &e, const States &b)
    {
#pragma unroll
        for (int j = 0; j < P; ++j) v[j] = fma2(e.v[j], v[j], b.v[j]);
    }
    __device__ __forceinline__ float dot(const States &c) const
    {
        uint64_t t = mul2(v[0], c.v[0]);
#pragma unroll
        for (int j = 1; j < P; ++j) t = fma2(v[j], c.v[j], t);
        float x, y;
        unpack2(t, x, y);
        return x + y;
    }
    __device__ __forceinline__ void set(int j, float f)
    {
        float x, y;
        unpack2(v[j / 2], x, y);
        v[j / 2] = j % 2 ? pack2(x, f) : pack2(f, y);
    }
    __device__ __forceinline__ float get(int j) const
    {
        float x, y;
        unpack2(v[j / 2], x, y);
        return j % 2 ? y : x;
    }
};
template <> struct States<1> {
    float v;
    __device__ __forceinline__ void load(const float *p) { v = *p; }
    __device__ __forceinline__ void scale(float f) { v *= f; }
    __device__ __forceinline__ void decay(float f, const States &a) { v = ex2(f * a.v); }
    __device__ __forceinline__ void advance(const States &e, const States &b) { v = fmaf(e.v, v, b.v); }
    __device__ __forceinline__ float dot(const States &c) const { return v * c.v; }
    __device__ __forceinline__ void set(int, float f) { v = f; }
    __device__ __forceinline__ float get(int) const { return v; }
};

// NS: states a thread carries; LG: log2 of the threads that share a channel.  U tokens go through the state at a
// time; their partial sums are then exchanged so that each of the channel's threads finishes tokens of its own.
template <typename T, typename TO, int NS, int LG>
__global__ void __launch_bounds__(kScanThreads) scan_kernel(const wr_rows rw, const wr_scan_args a)
{
    constexpr uint32_t TPC = 1u << LG, CB = kScanThreads >> LG, HELD = NS * TPC;            // channels per block, states held
    constexpr uint32_t BST = (HELD + 3) & ~3u;                                              // a token's B (or C) in shared memory
    constexpr uint32_t TILE = HELD > 128 ? 16 : 32;                                         // tokens per stage
    constexpr int LU = LG < 2 ? 2 : LG > 4 ? 4 : LG, U = NS > 4 ? 4 : 1 << LU, KEEP = U > (int)TPC ? U / (int)TPC : 1;
    extern __shared__ __align__(16) uint8_t sm_scan[];
    float *bs = reinterpret_cast<float *>(sm_scan), *cs = bs + 2 * TILE * BST;              // [2][TILE][BST]
    float *dts = cs + 2 * TILE * BST, *ys = dts + 2 * TILE * CB;                            // [2][TILE][CB], [TILE][CB]
    T *xs = reinterpret_cast<T *>(ys + TILE * CB), *zs = xs + 2 * TILE * CB;
    pdl_trigger();
    const uint32_t seq = blockIdx.y, tid = threadIdx.x;
    const uint32_t c_base = blockIdx.x * CB, cl = tid >> LG, part = tid & (TPC - 1), c = c_base + cl;
    const uint32_t ld = wr_ld(a.inner), lds = wr_ld(a.state), bc4 = (a.state + 3) / 4;      // 4-value pieces per token
    if (BST > 4 * bc4)
        for (uint32_t i = tid; i < 4 * TILE * BST; i += kScanThreads) bs[i] = 0.f;          // (B and C beyond `state`)
    States<NS> A2, S;
#pragma unroll
    for (int j = 0; j < NS; ++j) {
        const uint32_t n = part * NS + j;
        A2.set(j, (c < a.inner && n < a.state) ? a.a2[(size_t)c * lds + n] : 0.f);
    }
    const float D = c < a.inner ? a.d[c] : 0.f;
    pdl_wait();
    const wr_seq_dev s = rw.seqs[seq];
    const uint32_t row0 = row0_of(rw, seq), n_tok = s.n;
    const float *st_in = reinterpret_cast<const float *>(s.st_in + a.state_off);
#pragma unroll
    for (int j = 0; j < NS; ++j) {
        const uint32_t n = part * NS + j;
        S.set(j, (!s.fresh && c < a.inner && n < a.state) ? st_in[(size_t)c * a.state + n] : 0.f);
    }
    __syncthreads();
    auto request = [&](uint32_t tile) {
        const uint32_t st = tile & 1, t0 = tile * TILE, nt = min(TILE, n_tok - t0);
        for (uint32_t i = tid; i < nt * (CB / 4); i += kScanThreads) {
            const uint32_t t = i / (CB / 4), q = i % (CB / 4), ch = c_base + 4 * q;
            if (ch >= ld) continue;
            const size_t row = row0 + t0 + t;
            const uint32_t at = (st * TILE + t) * CB + 4 * q;
            cp_async<4 * sizeof(T)>(xs + at, static_cast<const T *>(a.x) + row * a.x_ld + ch);
            cp_async<4 * sizeof(T)>(zs + at, static_cast<const T *>(a.z) + row * a.z_ld + ch);
            cp_async<16>(dts + at, a.dt + row * ld + ch);
        }
        for (uint32_t i = tid; i < nt * bc4; i += kScanThreads) {
            const uint32_t t = i / bc4, q = i % bc4;
            const float *src = a.bc + (size_t)(row0 + t0 + t) * a.bc_ld + 4 * q;
            cp_async<16>(bs + (st * TILE + t) * BST + 4 * q, src + a.b_off);
            cp_async<16>(cs + (st * TILE + t) * BST + 4 * q, src + a.c_off);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const uint32_t tiles = (n_tok + TILE - 1) / TILE;
    request(0);
    for (uint32_t tile = 0; tile < tiles; ++tile) {
        const uint32_t st = tile & 1, t0 = tile * TILE, nt = min(TILE, n_tok - t0);
        if (tile + 1 < tiles) {
            request(tile + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        // What NT tokens bring, worked out one group ahead of the state's chain: decays, dt x B, C
        constexpr int NT = U / 2;
        struct Group { States<NS> e[NT], b[NT], c[NT]; };
        auto fetch = [&](Group &g, uint32_t t0, auto n_tokens) {
#pragma unroll
            for (int i = 0; i < decltype(n_tokens)::value; ++i) {
                const uint32_t t = st * TILE + t0 + i;
                const float dt = dts[t * CB + cl], dx = dt * to_f32(xs[t * CB + cl]);
                g.b[i].load(bs + t * BST + part * NS);
                g.c[i].load(cs + t * BST + part * NS);
                g.e[i].decay(dt, A2);
                g.b[i].scale(dx);
            }
        };
        float y[U];
        auto chain = [&](const Group &g, int i, int u) {
            S.advance(g.e[i], g.b[i]);
            y[u] = S.dot(g.c[i]);
        };
        // the channel's threads exchange their parts of U tokens' sums and finish some tokens each
        auto finish = [&](uint32_t tb) {
            uint32_t first = 0, width = U;                       // this thread keeps tokens [first, first + width)
#pragma unroll
            for (uint32_t o = 1; o < TPC; o <<= 1) {
                if (width > 1) {
                    const uint32_t half = width / 2;
                    const bool upper = (part & o) != 0;
#pragma unroll
                    for (int i = 0; i < U / 2; ++i) {
                        if (i < (int)half) {
                            const float send = upper ? y[i] : y[i + half], own = upper ? y[i + half] : y[i];
                            y[i] = own + __shfl_xor_sync(0xffffffffu, send, o);
                        }
                    }
                    if (upper) first += half;
                    width = half;
                } else {
                    y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
                }
            }
#pragma unroll
            for (int i = 0; i < KEEP; ++i) {
                const uint32_t t = tb + first + i, at = (st * TILE + t) * CB + cl;
                if (t < nt && part < (uint32_t)U) {
                    const float v = fmaf(D, to_f32(xs[at]), y[i]) * siluf(to_f32(zs[at]));
                    ys[t * CB + cl] = c < a.inner ? v : 0.f;
                }
            }
        };
        Group ga, gb;
        if (nt == TILE) {
            using All = std::integral_constant<int, NT>;
            fetch(ga, 0, All());
#pragma unroll 1
            for (uint32_t tb = 0; tb < TILE; tb += U) {
                fetch(gb, tb + NT, All());
#pragma unroll
                for (int i = 0; i < NT; ++i) chain(ga, i, i);
                if (tb + U < TILE) fetch(ga, tb + U, All());
#pragma unroll
                for (int i = 0; i < NT; ++i) chain(gb, i, NT + i);
                finish(tb);
            }
        } else {
#pragma unroll 1
            for (uint32_t tb = 0; tb < nt; tb += U) {
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    y[u] = 0.f;
                    if (tb + u < nt) {
                        fetch(ga, tb + u, std::integral_constant<int, 1>());
                        chain(ga, 0, u);
                    }
                }
                finish(tb);
            }
        }
        __syncthreads();
        for (uint32_t i = tid; i < nt * (CB / 4); i += kScanThreads) {
            const uint32_t t = i / (CB / 4), q = i % (CB / 4), ch = c_base + 4 * q;
            if (ch < ld) Out<TO>(a.out, row0 + t0 + t, ld).put4(ch, load4(ys + t * CB + 4 * q));
        }
    }
    float *st_out = reinterpret_cast<float *>(s.st_out + a.state_off);
#pragma unroll
    for (int j = 0; j < NS; ++j) {
        const uint32_t n = part * NS + j;
        if (c < a.inner && n < a.state) st_out[(size_t)c * a.state + n] = S.get(j);
    }
}

// One token per session (a decode step): four states per thread straight from memory, nothing staged.
constexpr uint32_t kStepThreads = 256;

template <typename TO, int LG>
__global__ void __launch_bounds__(kStepThreads) scan_step_kernel(const wr_rows rw, const wr_scan_args a)
{
    constexpr uint32_t TPC = 1u << LG;
    pdl_trigger();
    const uint32_t seq = blockIdx.y, part = threadIdx.x & (TPC - 1), c = (blockIdx.x * kStepThreads + threadIdx.x) >> LG;
    const uint32_t ld = wr_ld(a.inner), lds = wr_ld(a.state);
    const bool in = c < a.inner;
    float4 a2 = make_float4(0.f, 0.f, 0.f, 0.f);
    const uint32_t n0 = 4 * part;
    if (in && n0 < lds) a2 = load4(a.a2 + (size_t)c * lds + n0);
    const float D = in ? a.d[c] : 0.f;
    pdl_wait();
    const wr_seq_dev s = rw.seqs[seq];
    float y = 0.f, x = 0.f, z = 0.f;
    if (in) {
        const float *from = reinterpret_cast<const float *>(s.st_in + a.state_off) + (size_t)c * a.state + n0;
        float *to = reinterpret_cast<float *>(s.st_out + a.state_off) + (size_t)c * a.state + n0;
        const float *bc = a.bc + (size_t)seq * a.bc_ld + n0;
        x = static_cast<const float *>(a.x)[(size_t)seq * a.x_ld + c];
        z = static_cast<const float *>(a.z)[(size_t)seq * a.z_ld + c];
        const float dt = a.dt[(size_t)seq * ld + c], dx = dt * x;
        const uint32_t left = n0 < a.state ? a.state - n0 : 0u;
        float S[4] = {0.f, 0.f, 0.f, 0.f};
        if (!s.fresh) {
            if (left >= 4 && a.state % 4 == 0) {
                const float4 v = load4(from);
                S[0] = v.x; S[1] = v.y; S[2] = v.z; S[3] = v.w;
            } else {
#pragma unroll
                for (uint32_t j = 0; j < 4; ++j)
                    if (j < left) S[j] = from[j];
            }
        }
        float4 b = make_float4(0.f, 0.f, 0.f, 0.f), cc = b;
        if (left) {
            b = load4(bc + a.b_off);
            cc = load4(bc + a.c_off);
        }
        S[0] = fmaf(ex2(dt * a2.x), S[0], dx * b.x);
        S[1] = fmaf(ex2(dt * a2.y), S[1], dx * b.y);
        S[2] = fmaf(ex2(dt * a2.z), S[2], dx * b.z);
        S[3] = fmaf(ex2(dt * a2.w), S[3], dx * b.w);
        y = fmaf(S[3], cc.w, fmaf(S[2], cc.z, fmaf(S[1], cc.y, S[0] * cc.x)));
        if (left >= 4 && a.state % 4 == 0) {
            store4(to, make_float4(S[0], S[1], S[2], S[3]));
        } else {
#pragma unroll
            for (uint32_t j = 0; j < 4; ++j)
                if (j < left) to[j] = S[j];
        }
    }
#pragma unroll
    for (uint32_t o = TPC >> 1; o >= 1; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (part == 0 && c < ld) Out<TO>(a.out, seq, ld).put(c, in ? fmaf(D, x, y) * siluf(z) : 0.f);
}

template <typename TO, int LG> int scan_step_one(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_scan_args &a)
{
    const dim3 grid(((wr_ld(a.inner) << LG) + kStepThreads - 1) / kStepThreads, rw.n_seq);
    WR_CUDA_TRY(wr_launch_pdl(scan_step_kernel<TO, LG>, grid, dim3(kStepThreads), 0, ctx->stream, rw, a));
    return finish_launch(ctx);
}
template <typename TO> int scan_step(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_scan_args &a)
{
    if (a.state <= 4) return scan_step_one<TO, 0>(ctx, rw, a);
    if (a.state <= 8) return scan_step_one<TO, 1>(ctx, rw, a);
    if (a.state <= 16) return scan_step_one<TO, 2>(ctx, rw, a);
    if (a.state <= 32) return scan_step_one<TO, 3>(ctx, rw, a);
    if (a.state <= 64) return scan_step_one<TO, 4>(ctx, rw, a);
    return scan_step_one<TO, 5>(ctx, rw, a);                     // (128 states at most)
}

template <typename T, typename TO, int NS, int LG> int scan_one(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_scan_args &a)
{
    constexpr uint32_t CB = kScanThreads >> LG, HELD = NS << LG, BST = (HELD + 3) & ~3u, TILE = HELD > 128 ? 16 : 32;
    constexpr size_t smem = (size_t)(4 * TILE * BST + 3 * TILE * CB) * 4 + (size_t)4 * TILE * CB * sizeof(T);
    auto k = scan_kernel<T, TO, NS, LG>;
    if (smem > 48 * 1024)
        WR_CUDA_TRY(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    WR_CUDA_TRY(wr_launch_pdl(k, dim3((wr_ld(a.inner) + CB - 1) / CB, rw.n_seq), dim3(kScanThreads), smem, ctx->stream, rw, a));
    return finish_launch(ctx);
}

// One state per thread while that is what it takes to fill the device, two above; a choice by the model's sizes
// alone, so that a session's sums are added in one order whatever the step looks like.
template <typename T, typename TO> int scan_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_scan_args &a)
{
    const bool few = (uint64_t)a.inner * a.state < 131072;
    if (a.state <= 1) return scan_one<T, TO, 1, 0>(ctx, rw, a);
    if (a.state <= 2) return scan_one<T, TO, 1, 1>(ctx, rw, a);
    if (a.state <= 4) return scan_one<T, TO, 1, 2>(ctx, rw, a);
    if (a.state <= 8) return scan_one<T, TO, 1, 3>(ctx, rw, a);
    if (a.state <= 16) return few ? scan_one<T, TO, 1, 4>(ctx, rw, a) : scan_one<T, TO, 2, 3>(ctx, rw, a);
    if (a.state <= 32) return few ? scan_one<T, TO, 1, 5>(ctx, rw, a) : scan_one<T, TO, 2, 4>(ctx, rw, a);
    if (a.state <= 64) return scan_one<T, TO, 2, 5>(ctx, rw, a);
    if (a.state <= 128) return scan_one<T, TO, 4, 5>(ctx, rw, a);
    if (a.state <= 256) return scan_one<T, TO, 8, 5>(ctx, rw, a);
    if (a.state <= 512) return scan_one<T, TO, 16, 5>(ctx, rw, a);
    return WR_CUDA_ERR_LIMIT;
}

// ------------------------------------------------------------- around attention

// Queries out of the projection row (scale and temperature applied), K and V into the session's pages.  The row's
// queries, keys and values are one list of pieces of W values; the blocks of grid.y share it.
template <typename TI, typename TQ, int W>
__global__ void __launch_bounds__(256) attn_prep_kernel(const wr_rows rw, const wr_attn_prep_args a)
{
    pdl_trigger();
    pdl_wait();
    const uint32_t row = blockIdx.x;
    const wr_seq_dev s = rw.seqs[seq_of(rw, row)];
    const uint32_t pos = s.pos + tok_of(rw, row);
    const wr_attn_geom g = a.g;
    const TI *in = static_cast<const TI *>(a.qkv) + (size_t)row * a.ld;
    float mul = a.scale;
    if (a.temp_every) mul *= 1.0f + a.temp_coef * logf((float)((pos + 1u) / a.temp_every + 1u));
    const uint32_t qs = g.q_stride(), kw = g.maps * g.kd;
    const uint32_t nq = g.vq() * qs / W, nk = g.n_kv * kw / W, nv = g.n_kv * g.vd / W;
    TQ *q = static_cast<TQ *>(a.q) + (size_t)row * g.vq() * qs;
    char *page = reinterpret_cast<char *>(s.pages[(size_t)g.layer * s.n_pages + pos / kPageTokens]);
    const uint32_t tok = pos % kPageTokens;
    for (uint32_t i = blockIdx.y * 256 + threadIdx.x; i < nq + nk + nv; i += gridDim.y * 256) {
        float v[W];
        auto fetch = [&](const TI *p) {
            if constexpr (W == 8) load8v(p, v);
            else v[0] = to_f32(*p);
        };
        if (i < nq) {
            const uint32_t at = i * W, vq = at / qs, e = at % qs, off = g.hd128 ? (vq % g.maps) * g.kd : 0u;   // the map's part of the row
            if (e >= off && e < off + g.kd) {
                fetch(in + vq * g.kd + e - off);
#pragma unroll
                for (int j = 0; j < W; ++j) v[j] *= mul;
            } else {
#pragma unroll
                for (int j = 0; j < W; ++j) v[j] = 0.f;
            }
            if constexpr (W == 8) store8v(q + at, v);
            else q[at] = from_f32<TQ>(v[0]);
            continue;
        }
        const uint32_t which = i < nq + nk ? 0u : 1u, at = (i - nq - which * nk) * W, dim = which ? g.vd : kw;
        fetch(in + (which ? a.v_off : a.k_off) + at);
        char *p = page + wr_geom_off(g.kv, at / dim, which, tok, at % dim);
        if constexpr (W == 8) {
            if (g.kv.elem == WR_CUDA_F32) store8v(reinterpret_cast<float *>(p), v);
            else store8v(reinterpret_cast<__half *>(p), v);
        } else {
            if (g.kv.elem == WR_CUDA_F32) *reinterpret_cast<float *>(p) = v[0];
            else *reinterpret_cast<__half *>(p) = from_f32<__half>(v[0]);
        }
    }
}

template <typename TI, typename TQ> cudaError_t prep_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_attn_prep_args &a)
{
    const wr_attn_geom &g = a.g;
    const uint32_t w = g.kd % 8 == 0 && g.vd % 8 == 0 ? 8 : 1;
    const uint32_t items = (g.vq() * g.q_stride() + g.n_kv * (g.maps * g.kd + g.vd)) / w;
    const dim3 grid(rw.n_rows, rw.n_rows <= WR_CUDA_BATCH_MAX ? (items + 255) / 256 : (items + 1023) / 1024), block(256);
    if (w == 8) return wr_launch_pdl(attn_prep_kernel<TI, TQ, 8>, grid, block, 0, ctx->stream, rw, a);
    return wr_launch_pdl(attn_prep_kernel<TI, TQ, 1>, grid, block, 0, ctx->stream, rw, a);
}

// One warp per query head: combine the maps, norm over the head, gate.
template <typename TG, typename TO>
__global__ void __launch_bounds__(256) attn_finish_kernel(const wr_rows rw, const wr_attn_finish_args a)
{
    pdl_trigger();
    pdl_wait();
    const wr_attn_geom g = a.g;
    const uint32_t row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, os = g.o_stride();
    const uint32_t n_out = g.n_q * g.vd, ld = wr_ld(n_out);
    const Out<TO> out(a.out, row, ld);
    for (uint32_t h = blockIdx.y * 8 + warp; h < g.n_q; h += gridDim.y * 8) {
        const float *o1 = a.o + ((size_t)row * g.vq() + h * g.maps) * os, *o2 = o1 + os;
        if (g.vd <= 128 && g.vd % 4 == 0) {                      // a lane's four values stay in registers
            const uint32_t i = 4 * lane;
            float4 d = make_float4(0.f, 0.f, 0.f, 0.f), gt = d;
            if (i < g.vd) {
                d = load4(o1 + i);
                if (a.gate) gt = load4(static_cast<const TG *>(a.gate) + (size_t)row * a.gate_ld + h * g.vd + i);
                if (g.maps == 2) {
                    const float4 e = load4(o2 + i);
                    d = make_float4(fmaf(-a.lambda, e.x, d.x), fmaf(-a.lambda, e.y, d.y), fmaf(-a.lambda, e.z, d.z),
                                    fmaf(-a.lambda, e.w, d.w));
                }
            }
            float k = 1.0f;
            if (g.maps == 2) {
                const float ss = fmaf(d.w, d.w, fmaf(d.z, d.z, fmaf(d.y, d.y, d.x * d.x)));
                k = (1.0f - a.diff_init) / sqrtf(warp_sum(ss) / (float)g.vd + a.eps);
            }
            if (i < g.vd) {
                d = make_float4(d.x * k, d.y * k, d.z * k, d.w * k);
                if (a.gate)
                    d = make_float4(d.x * sigmoidf(gt.x), d.y * sigmoidf(gt.y), d.z * sigmoidf(gt.z), d.w * sigmoidf(gt.w));
                out.put4(h * g.vd + i, d);
            }
            continue;
        }
        float k = 1.0f;
        if (g.maps == 2) {
            float ss = 0.f;
            for (uint32_t i = lane; i < g.vd; i += 32) {
                const float d = fmaf(-a.lambda, o2[i], o1[i]);
                ss = fmaf(d, d, ss);
            }
            k = (1.0f - a.diff_init) / sqrtf(warp_sum(ss) / (float)g.vd + a.eps);
        }
        for (uint32_t i = lane; i < g.vd; i += 32) {
            float v = g.maps == 2 ? fmaf(-a.lambda, o2[i], o1[i]) * k : o1[i];
            if (a.gate)
                v *= sigmoidf(to_f32(static_cast<const TG *>(a.gate)[(size_t)row * a.gate_ld + h * g.vd + i]));
            out.put(h * g.vd + i, v);
        }
    }
    if (blockIdx.y == 0 && threadIdx.x < ld - n_out) out.put(n_out + threadIdx.x, 0.f);
}

// --------------------------------------------- attention over any cache layout

__device__ __forceinline__ void load8(const char *p, uint32_t elem, float (&v)[8])
{
    if (elem == WR_CUDA_F32) {
        const float4 a = *reinterpret_cast<const float4 *>(p), b = *reinterpret_cast<const float4 *>(p + 16);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    } else {
        const uint4 u = *reinterpret_cast<const uint4 *>(p);
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __half22float2(*reinterpret_cast<const __half2 *>(&w[i]));
            v[2 * i] = f.x;
            v[2 * i + 1] = f.y;
        }
    }
}

// Columns [d0, d0 + dims) of rows [key0, key0 + n_keys) of a head's K or V into shared memory (row stride `stride`).
__device__ __forceinline__ void stage_rows(const uint64_t *table, const wr_kv_geom &g, uint32_t head, uint32_t which,
                                           uint32_t key0, uint32_t n_keys, uint32_t d0, uint32_t dims, float *dst,
                                           uint32_t stride)
{
    const uint32_t lo8 = d0 / 8u, n8 = (d0 + dims + 7u) / 8u - lo8;
    for (uint32_t i = threadIdx.x; i < n_keys * n8; i += blockDim.x) {
        const uint32_t k = i / n8, d = (lo8 + i % n8) * 8u, key = key0 + k;
        const char *p = reinterpret_cast<const char *>(table[key / kPageTokens]) +
                        wr_geom_off(g, head, which, key % kPageTokens, d);
        float v[8];
        load8(p, g.elem, v);
#pragma unroll
        for (int e = 0; e < 8; ++e)
            if (d + e >= d0 && d + e < d0 + dims) dst[k * stride + d + e - d0] = v[e];
    }
}

constexpr uint32_t kAnyRows = 32, kAnyKeys = 32, kAnyThreads = 128;

// Prompt rows: a block is 32 query rows of one query (head, map); four threads share a row.
template <int VC>
__global__ void __launch_bounds__(kAnyThreads) attn_rows_any_kernel(const wr_rows rw, const wr_attn_geom g,
                                                                    const float *q, float *out)
{
    extern __shared__ float sm_any[];
    const uint32_t ks = g.kd | 1u, vs = g.shared ? ks : g.vd;
    // P: [rows][33]; where the key's first columns are the value, one copy of the row serves both
    float *Q = sm_any, *K = Q + kAnyRows * ks, *P = K + kAnyKeys * ks, *V = g.shared ? K : P + kAnyRows * (kAnyKeys + 1);
    pdl_trigger();
    pdl_wait();
    const wr_seq_dev s = rw.seqs[0];
    const uint64_t *table = s.pages + (size_t)g.layer * s.n_pages;
    const uint32_t t0 = blockIdx.x * kAnyRows, vq = blockIdx.y, head = vq / g.maps / (g.n_q / g.n_kv), map = vq % g.maps;
    const uint32_t rows = min(kAnyRows, s.n - t0), r = threadIdx.x >> 2, sub = threadIdx.x & 3;
    for (uint32_t i = threadIdx.x; i < kAnyRows * g.kd; i += kAnyThreads) {
        const uint32_t rr = i / g.kd, d = i % g.kd;
        Q[rr * ks + d] = rr < rows ? q[((size_t)(t0 + rr) * g.vq() + vq) * g.kd + d] : 0.f;
    }
    const uint32_t my_pos = s.pos + t0 + r, key_end = s.pos + t0 + rows;
    float m = -INFINITY, l = 0.f, acc[VC];
#pragma unroll
    for (int i = 0; i < VC; ++i) acc[i] = 0.f;
    for (uint32_t k0 = 0; k0 < key_end; k0 += kAnyKeys) {
        const uint32_t nk = min(kAnyKeys, key_end - k0);
        __syncthreads();
        stage_rows(table, g.kv, head, 0, k0, nk, map * g.kd, g.kd, K, ks);
        if (!g.shared) stage_rows(table, g.kv, head, 1, k0, nk, 0, g.vd, V, vs);
        __syncthreads();
        float sc[kAnyKeys / 4], mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < (int)kAnyKeys / 4; ++i) {
            const uint32_t k = sub + 4 * i;
            sc[i] = -INFINITY;
            if (k < nk && k0 + k <= my_pos) {
                float d = 0.f;
                for (uint32_t e = 0; e < g.kd; ++e) d = fmaf(Q[r * ks + e], K[k * ks + e], d);
                sc[i] = d;
            }
            mx = fmaxf(mx, sc[i]);
        }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m, mx);                        // (key 0 is visible to every row: finite from the start)
        const float corr = expf(m - m_new);
        float ps = 0.f;
#pragma unroll
        for (int i = 0; i < (int)kAnyKeys / 4; ++i) {
            const float p = expf(sc[i] - m_new);
            P[r * (kAnyKeys + 1) + sub + 4 * i] = p;
            ps += p;
        }
        ps += __shfl_xor_sync(0xffffffffu, ps, 1);
        ps += __shfl_xor_sync(0xffffffffu, ps, 2);
        l = fmaf(l, corr, ps);
        m = m_new;
        __syncwarp();
#pragma unroll
        for (int i = 0; i < VC; ++i) acc[i] *= corr;
        for (uint32_t k = 0; k < nk; ++k) {
            const float p = P[r * (kAnyKeys + 1) + k];
#pragma unroll
            for (int i = 0; i < VC; ++i) {
                const uint32_t c = sub + 4 * i;
                if (c < g.vd) acc[i] = fmaf(p, V[k * vs + c], acc[i]);
            }
        }
    }
    if (r < rows) {
        const float inv = 1.0f / l;
        float *o = out + ((size_t)(t0 + r) * g.vq() + vq) * g.vd;
#pragma unroll
        for (int i = 0; i < VC; ++i) {
            const uint32_t c = sub + 4 * i;
            if (c < g.vd) o[c] = acc[i] * inv;
        }
    }
}

// Decode: a block is one chunk of keys of one (session, kv head) for all of the head's queries.  Partial rows
// (m, l, o[vd]) go to ws[session][vq][chunk]; attn_merge_any_kernel adds them up in chunk order.  A head with many
// queries is served by `parts` blocks of `per` queries each.
constexpr uint32_t kChunkKeys = 256;

__host__ __device__ inline uint32_t any_ws_stride(uint32_t vd) { return vd + 2u; }

__global__ void __launch_bounds__(kAnyThreads) attn_chunk_any_kernel(const wr_rows rw, const wr_attn_geom g,
                                                                     const float *q, float *ws, uint32_t chunks,
                                                                     uint32_t parts, uint32_t per)
{
    extern __shared__ float sm_any[];
    const uint32_t group = g.n_q / g.n_kv * g.maps, kw = g.maps * g.kd, ks = kw | 1u;
    const uint32_t head = blockIdx.y / parts, v_lo = blockIdx.y % parts * per, nq = min(per, group - v_lo);
    float *Q = sm_any, *K = Q + nq * g.kd, *S = K + kAnyKeys * ks, *M = S + nq * kChunkKeys, *L = M + nq;
    pdl_trigger();
    pdl_wait();
    const uint32_t chunk = blockIdx.x, seq = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const wr_seq_dev s = rw.seqs[seq];
    const uint32_t len = s.pos + 1, lo = chunk * kChunkKeys;
    if (lo >= len) return;
    const uint32_t n = min(kChunkKeys, len - lo);
    const uint64_t *table = s.pages + (size_t)g.layer * s.n_pages;
    const float *qrow = q + ((size_t)seq * g.vq() + head * group + v_lo) * g.kd;
    for (uint32_t i = threadIdx.x; i < nq * g.kd; i += kAnyThreads) Q[i] = qrow[i];
    for (uint32_t k0 = 0; k0 < n; k0 += kAnyKeys) {
        const uint32_t nk = min(kAnyKeys, n - k0);
        __syncthreads();
        stage_rows(table, g.kv, head, 0, lo + k0, nk, 0, kw, K, ks);
        __syncthreads();
        for (uint32_t i = threadIdx.x; i < nq * kAnyKeys; i += kAnyThreads) {
            const uint32_t v = i / kAnyKeys, k = i % kAnyKeys;
            if (k >= nk) continue;
            const float *kr = K + k * ks + ((v_lo + v) % g.maps) * g.kd, *qr = Q + v * g.kd;
            float d = 0.f;
            for (uint32_t e = 0; e < g.kd; ++e) d = fmaf(qr[e], kr[e], d);
            S[v * kChunkKeys + k0 + k] = d;
        }
    }
    __syncthreads();
    for (uint32_t v = warp; v < nq; v += kAnyThreads / 32) {
        float mx = -INFINITY, sum = 0.f;
        for (uint32_t k = lane; k < n; k += 32) mx = fmaxf(mx, S[v * kChunkKeys + k]);
#pragma unroll
        for (int o = 16; o >= 1; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        for (uint32_t k = lane; k < n; k += 32) {
            const float p = expf(S[v * kChunkKeys + k] - mx);
            S[v * kChunkKeys + k] = p;
            sum += p;
        }
        sum = warp_sum(sum);
        if (lane == 0) { M[v] = mx; L[v] = sum; }
    }
    __syncthreads();
    const uint32_t stride = any_ws_stride(g.vd);
    constexpr uint32_t B = 8;
    for (uint32_t c = threadIdx.x; c < g.vd; c += kAnyThreads)
        for (uint32_t v0 = 0; v0 < nq; v0 += B) {
            float acc[B];
#pragma unroll
            for (uint32_t j = 0; j < B; ++j) acc[j] = 0.f;
            for (uint32_t k = 0; k < n; ++k) {
                const uint32_t key = lo + k;
                const char *p = reinterpret_cast<const char *>(table[key / kPageTokens]) +
                                wr_geom_off(g.kv, head, g.shared ? 0u : 1u, key % kPageTokens, c);
                const float x = g.kv.elem == WR_CUDA_F32 ? *reinterpret_cast<const float *>(p)
                                                         : __half2float(*reinterpret_cast<const __half *>(p));
#pragma unroll
                for (uint32_t j = 0; j < B; ++j)
                    if (v0 + j < nq) acc[j] = fmaf(S[(v0 + j) * kChunkKeys + k], x, acc[j]);
            }
#pragma unroll
            for (uint32_t j = 0; j < B; ++j)
                if (v0 + j < nq)
                    ws[(((size_t)seq * g.vq() + head * group + v_lo + v0 + j) * chunks + chunk) * stride + 2 + c] = acc[j];
        }
    for (uint32_t v = threadIdx.x; v < nq; v += kAnyThreads) {
        float *w = ws + (((size_t)seq * g.vq() + head * group + v_lo + v) * chunks + chunk) * stride;
        w[0] = M[v];
        w[1] = L[v];
    }
}

__global__ void __launch_bounds__(128) attn_merge_any_kernel(const wr_rows rw, const wr_attn_geom g, const float *ws,
                                                             float *out, uint32_t chunks)
{
    pdl_trigger();
    pdl_wait();
    const uint32_t vq = blockIdx.x, seq = blockIdx.y;
    const uint32_t n = (rw.seqs[seq].pos + 1 + kChunkKeys - 1) / kChunkKeys, stride = any_ws_stride(g.vd);
    const float *w = ws + ((size_t)seq * g.vq() + vq) * chunks * stride;
    float m = -INFINITY, l = 0.f;
    for (uint32_t i = 0; i < n; ++i) m = fmaxf(m, w[(size_t)i * stride]);
    for (uint32_t i = 0; i < n; ++i) l = fmaf(w[(size_t)i * stride + 1], expf(w[(size_t)i * stride] - m), l);
    for (uint32_t c = threadIdx.x; c < g.vd; c += 128) {
        float o = 0.f;
        for (uint32_t i = 0; i < n; ++i) o = fmaf(w[(size_t)i * stride + 2 + c], expf(w[(size_t)i * stride] - m), o);
        out[((size_t)seq * g.vq() + vq) * g.vd + c] = o / l;
    }
}

template <int VC> int rows_any(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_attn_geom &g, const float *q, float *out)
{
    const size_t smem = (size_t)(2 * kAnyRows * (g.kd | 1u) + (g.shared ? 0u : kAnyKeys * g.vd) + kAnyRows * (kAnyKeys + 1)) * 4;
    int rc = allow_smem(attn_rows_any_kernel<VC>, smem);
    if (rc != WR_CUDA_OK) return rc;
    WR_CUDA_TRY(wr_launch_pdl(attn_rows_any_kernel<VC>, dim3((rw.n_rows + kAnyRows - 1) / kAnyRows, g.vq()),
                              dim3(kAnyThreads), smem, ctx->stream, rw, g, q, out));
    return finish_launch(ctx);
}

}  // namespace

int wr_embed_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const uint32_t *tokens, const void *table, int table_type,
                    const double *turns, float *x, uint32_t width, float scale)
{
    const dim3 grid((wr_ld(width) + 511) / 512, rw.n_rows);
    if (table_type == WR_ACT_BF16)
        embed_kernel<__nv_bfloat16><<<grid, 256, 0, ctx->stream>>>(rw, tokens, (const __nv_bfloat16 *)table, turns, x, width, scale);
    else
        embed_kernel<float><<<grid, 256, 0, ctx->stream>>>(rw, tokens, (const float *)table, turns, x, width, scale);
    return finish_launch(ctx);
}

int wr_group_norm_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_norm_args &a)
{
    cudaError_t e = cudaSuccess;
    if (a.out_type == WR_ACT_BF16) e = norm_launch<__nv_bfloat16>(ctx, rw, a);
    else if (a.out_type == WR_ACT_SPLIT) e = norm_launch<Split>(ctx, rw, a);
    else e = norm_launch<float>(ctx, rw, a);
    WR_CUDA_TRY(e);
    return finish_launch(ctx);
}

int wr_polynorm_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_polynorm_args &a)
{
    const dim3 grid(rw.n_rows), block(kPolyThreads);
    if (a.z_type == WR_ACT_BF16)
        WR_CUDA_TRY(wr_launch_pdl(polynorm_kernel<__nv_bfloat16, __nv_bfloat16>, grid, block, 0, ctx->stream, a));
    else if (a.out_type == WR_ACT_SPLIT)
        WR_CUDA_TRY(wr_launch_pdl(polynorm_kernel<float, Split>, grid, block, 0, ctx->stream, a));
    else
        WR_CUDA_TRY(wr_launch_pdl(polynorm_kernel<float, float>, grid, block, 0, ctx->stream, a));
    return finish_launch(ctx);
}

int wr_conv_silu_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_conv_args &a)
{
    WR_CUDA_TRY(a.type == WR_ACT_BF16 ? conv_launch<__nv_bfloat16>(ctx, rw, a) : conv_launch<float>(ctx, rw, a));
    return finish_launch(ctx);
}

int wr_scan_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_scan_args &a)
{
    if (rw.decode && a.type == WR_ACT_F32 && a.state <= 128)
        return a.out_type == WR_ACT_SPLIT ? scan_step<Split>(ctx, rw, a) : scan_step<float>(ctx, rw, a);
    if (a.type == WR_ACT_BF16) return scan_launch<__nv_bfloat16, __nv_bfloat16>(ctx, rw, a);
    return a.out_type == WR_ACT_SPLIT ? scan_launch<float, Split>(ctx, rw, a) : scan_launch<float, float>(ctx, rw, a);
}

int wr_attn_prep_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_attn_prep_args &a)
{
    const bool half_in = a.type == WR_ACT_F16, half_q = a.q_type == WR_ACT_F16;
    WR_CUDA_TRY(half_in ? (half_q ? prep_launch<__half, __half>(ctx, rw, a) : prep_launch<__half, float>(ctx, rw, a))
                        : (half_q ? prep_launch<float, __half>(ctx, rw, a) : prep_launch<float, float>(ctx, rw, a)));
    return finish_launch(ctx);
}

int wr_attn_any_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_attn_geom &g, const float *q, float *out,
                       uint32_t max_len)
{
    if (!rw.decode) {
        if (g.vd <= 64) return rows_any<16>(ctx, rw, g, q, out);
        if (g.vd <= 128) return rows_any<32>(ctx, rw, g, q, out);
        if (g.vd <= 256) return rows_any<64>(ctx, rw, g, q, out);
        if (g.vd <= 512) return rows_any<128>(ctx, rw, g, q, out);
        return WR_CUDA_ERR_LIMIT;
    }
    const uint32_t group = g.n_q / g.n_kv * g.maps, chunks = (max_len + kChunkKeys - 1) / kChunkKeys;
    int rc = wr_ctx_reserve_ws(ctx, (size_t)rw.n_seq * g.vq() * chunks * any_ws_stride(g.vd) * sizeof(float), 0);
    if (rc != WR_CUDA_OK) return rc;
    auto bytes = [&](uint32_t nq) {
        return (size_t)(nq * g.kd + kAnyKeys * ((g.maps * g.kd) | 1u) + nq * kChunkKeys + 2 * nq) * 4;
    };
    uint32_t parts = 1;
    while (parts < group && bytes((group + parts - 1) / parts) > 200 * 1024) ++parts;
    const uint32_t per = (group + parts - 1) / parts;
    parts = (group + per - 1) / per;
    const size_t smem = bytes(per);
    rc = allow_smem(attn_chunk_any_kernel, smem);
    if (rc != WR_CUDA_OK) return rc;
    WR_CUDA_TRY(wr_launch_pdl(attn_chunk_any_kernel, dim3(chunks, g.n_kv * parts, rw.n_seq), dim3(kAnyThreads), smem,
                              ctx->stream, rw, g, q, ctx->ws, chunks, parts, per));
    rc = finish_launch(ctx);
    if (rc != WR_CUDA_OK) return rc;
    WR_CUDA_TRY(wr_launch_pdl(attn_merge_any_kernel, dim3(g.vq(), rw.n_seq), dim3(128), 0, ctx->stream, rw, g,
                              (const float *)ctx->ws, out, chunks));
    return finish_launch(ctx);
}

int wr_attn_finish_launch(wr_cuda_ctx *ctx, const wr_rows &rw, const wr_attn_finish_args &a)
{
    const dim3 grid(rw.n_rows, (a.g.n_q + 7) / 8), block(256);
    if (a.out_type == WR_ACT_BF16)
        WR_CUDA_TRY(wr_launch_pdl(attn_finish_kernel<__half, __nv_bfloat16>, grid, block, 0, ctx->stream, rw, a));
    else if (a.out_type == WR_ACT_SPLIT)
        WR_CUDA_TRY(wr_launch_pdl(attn_finish_kernel<float, Split>, grid, block, 0, ctx->stream, rw, a));
    else
        WR_CUDA_TRY(wr_launch_pdl(attn_finish_kernel<float, float>, grid, block, 0, ctx->stream, rw, a));
    return finish_launch(ctx);
}
