// model_glue.cu — the layer stack around attention, device-resident.
//
// The reference's decode body (src/core/session.c:405-568) runs, per layer:
// RMSNorm, the Q/K/V projections, per-head QK-norm, RoPE + KV append +
// attention, the output projection, a residual add, RMSNorm, the gate / up
// projections, SiLU(gate)*up, the down projection, a residual add; then the
// final RMSNorm and the LM head.  With attention on the GPU, leaving the rest
// on the host makes every layer cross the bus twice.  This file keeps a copy of
// the F32 weights on the device (wr_cuda_model) and runs the whole stack there:
// the rows of a forward pass enter as token ids and leave as logits.
//
// All arithmetic is F32, as the reference's F32 paths are (kernels.c:978-1090
// matmul with GGML-layout weights W[out][in]; :1276-1313 RMSNorm
// x * (1/sqrt(mean(x^2)+eps)) * w; :1318-1350 SiLU(a)*b).  Sums run in a
// different order than the host's SIMD loops, so results agree to F32 rounding,
// not bit for bit.  A row's result does not depend on how many other rows
// share the call (same lanes, same order), which keeps batched logits
// byte-equal to serial ones as the reference promises (src/core/batch.c:1-40).
//
// Kernels: a row-block GEMV (gemv.cu: each warp owns 1-4 weight rows, the activation
// rows sit in shared memory, the weights stream from HBM exactly once per group
// of up to 16 activation rows) with optional fused RMSNorm on the input, fused
// residual add or SiLU*up on the output; per-head RMSNorm; embedding gather;
// row RMSNorm; a two-step arg-max with the reference's tie rule (first maximum wins,
// src/cli/wayrt.c:805-812).
#include <math.h>
#include <stdlib.h>

#include <chrono>

#include "gemv.cuh"
#include "model.cuh"
#include "wr_internal.cuh"

namespace {

constexpr uint32_t kLogitRowsMax = WR_CUDA_BATCH_MAX;

// resid[r][:] = table[token[r]][:]
__global__ void embed_rows_kernel(const uint32_t *tokens, const float *table, float *out, uint32_t hidden)
{
    const float4 *src = reinterpret_cast<const float4 *>(table + (size_t)tokens[blockIdx.x] * hidden);
    float4 *dst = reinterpret_cast<float4 *>(out + (size_t)blockIdx.x * hidden);
    for (uint32_t i = threadIdx.x; i < hidden / 4; i += blockDim.x) dst[i] = src[i];
}

// In-place RMSNorm of every head vector: vectors [0, n_a) of `a`, then [0, n_b) of `b`; one warp each.
__global__ void head_rmsnorm_kernel(float *a, const float *wa, uint32_t n_a, float *b, const float *wb,
                                    uint32_t n_b, uint32_t dim, float eps)
{
    const uint32_t v = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (v >= n_a + n_b) return;
    float *x = (v < n_a) ? a + (size_t)v * dim : b + (size_t)(v - n_a) * dim;
    const float *w = (v < n_a) ? wa : wb;
    float ss = 0.f;
    for (uint32_t i = lane; i < dim; i += 32) ss += x[i] * x[i];
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = 1.0f / sqrtf(ss / (float)dim + eps);
    for (uint32_t i = lane; i < dim; i += 32) x[i] = x[i] * inv * w[i];
}

// out[r][:] = RMSNorm(x[r][:]) * w; one block per row
__global__ void rmsnorm_rows_kernel(const float *x, uint32_t x_stride, const float *w, float *out,
                                    uint32_t out_stride, uint32_t dim, float eps)
{
    __shared__ float part[32];
    const float *xr = x + (size_t)blockIdx.x * x_stride;
    float ss = 0.f;
    for (uint32_t i = threadIdx.x; i < dim; i += blockDim.x) ss += xr[i] * xr[i];
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
    __syncthreads();
    if (threadIdx.x < 32) {
        float t = (threadIdx.x < (blockDim.x >> 5)) ? part[threadIdx.x] : 0.f;
#pragma unroll
        for (int o = 16; o >= 1; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
        if (threadIdx.x == 0) part[0] = 1.0f / sqrtf(t / (float)dim + eps);
    }
    __syncthreads();
    const float inv = part[0];
    float *o_ = out + (size_t)blockIdx.x * out_stride;
    for (uint32_t i = threadIdx.x; i < dim; i += blockDim.x) o_[i] = xr[i] * inv * w[i];
}

// First maximum of each row (strict >, so the lowest id wins a tie), in two steps: kArgmaxParts
// blocks per row each reduce a slice of the vocabulary to (value, index); one warp per row then
// reduces the slices' results.  (value, index) pairs are compared as "greater value, or equal
// value and lower index", so the order of the reduction does not matter.
constexpr int kArgmaxParts = WR_ARGMAX_PARTS;

__device__ __forceinline__ bool argmax_better(float v, uint32_t i, float bv, uint32_t bi)
{
    return bi == 0xffffffffu || (i != 0xffffffffu && (v > bv || (v == bv && i < bi)));
}

__device__ __forceinline__ void argmax_warp(float &best, uint32_t &at)
{
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const uint32_t oi = __shfl_xor_sync(0xffffffffu, at, o);
        if (argmax_better(ov, oi, best, at)) { best = ov; at = oi; }
    }
}

__global__ void __launch_bounds__(256) argmax_parts_kernel(const float *logits, uint32_t ld, uint32_t vocab, float *part_v,
                                                           uint32_t *part_i)
{
    __shared__ float bv[8];
    __shared__ uint32_t bi[8];
    const uint32_t row = blockIdx.y, part = blockIdx.x;
    const uint32_t per = (vocab + kArgmaxParts - 1) / kArgmaxParts;
    const uint32_t lo = part * per, hi = min(lo + per, vocab);
    const float *r = logits + (size_t)row * ld;
    float best = -INFINITY;
    uint32_t at = 0xffffffffu;
    for (uint32_t i = lo + threadIdx.x; i < hi; i += blockDim.x) {
        const float v = r[i];
        if (argmax_better(v, i, best, at)) { best = v; at = i; }
    }
    argmax_warp(best, at);
    if ((threadIdx.x & 31) == 0) { bv[threadIdx.x >> 5] = best; bi[threadIdx.x >> 5] = at; }
    __syncthreads();
    if (threadIdx.x < 32) {
        best = threadIdx.x < 8 ? bv[threadIdx.x] : -INFINITY;
        at = threadIdx.x < 8 ? bi[threadIdx.x] : 0xffffffffu;
        argmax_warp(best, at);
        if (threadIdx.x == 0) {
            part_v[row * kArgmaxParts + part] = best;
            part_i[row * kArgmaxParts + part] = at;
        }
    }
}

__global__ void argmax_final_kernel(const float *part_v, const uint32_t *part_i, uint32_t *out)
{
    const uint32_t row = blockIdx.x, lane = threadIdx.x;
    float best = -INFINITY;
    uint32_t at = 0xffffffffu;
    for (uint32_t i = lane; i < (uint32_t)kArgmaxParts; i += 32) {
        const float v = part_v[row * kArgmaxParts + i];
        const uint32_t idx = part_i[row * kArgmaxParts + i];
        if (argmax_better(v, idx, best, at)) { best = v; at = idx; }
    }
    argmax_warp(best, at);
    if (lane == 0) out[row] = at;
}

}  // namespace

int wr_argmax_launch(cudaStream_t st, const float *logits, uint32_t ld, uint32_t vocab, uint32_t rows, float *part_v,
                     uint32_t *part_i, uint32_t *best)
{
    argmax_parts_kernel<<<dim3(kArgmaxParts, rows), 256, 0, st>>>(logits, ld, vocab, part_v, part_i);
    argmax_final_kernel<<<rows, 32, 0, st>>>(part_v, part_i, best);
    WR_CUDA_TRY(cudaGetLastError());
    return WR_CUDA_OK;
}

// ------------------------------------------------------------------ the model

namespace {

int gemv(wr_cuda_model *m, GemvParams &p, uint32_t n_total_for_width)
{
    ++m->launches;
    return wr_gemv_launch(m->ctx, p, n_total_for_width);
}

size_t up256(size_t n) { return (n + 255u) & ~(size_t)255u; }

}  // namespace

extern "C" int wr_cuda_model_create(wr_cuda_ctx *ctx, const wr_cuda_model_desc *d, wr_cuda_model **out)
{
    if (!ctx || !d || !out) return WR_CUDA_ERR_INVAL;
    *out = nullptr;
    if (d->n_layers == 0 || d->n_layers > WR_CUDA_MAX_LAYERS || !d->layers || !d->embed || !d->lm_head ||
        !d->final_norm || d->hidden == 0 || d->n_q_heads == 0 || d->n_kv_heads == 0 || d->head_dim == 0 ||
        d->vocab == 0 || d->max_rows == 0)
        return WR_CUDA_ERR_INVAL;
    // rows move as 16-byte vectors
    if ((d->hidden & 3u) || (d->head_dim & 3u)) return WR_CUDA_ERR_UNSUPPORTED;
    for (uint32_t L = 0; L < d->n_layers; ++L) {
        const wr_cuda_layer_desc &l = d->layers[L];
        if (!l.attn_norm || !l.wq || !l.wk || !l.wv || !l.wo || !l.ffn_norm || !l.w_gate || !l.w_up ||
            !l.w_down || l.ffn_dim == 0)
            return WR_CUDA_ERR_INVAL;
        if ((l.q_norm == nullptr) != (l.k_norm == nullptr)) return WR_CUDA_ERR_INVAL;
        if (l.ffn_dim & 3u) return WR_CUDA_ERR_UNSUPPORTED;
    }
    std::lock_guard<std::mutex> g(ctx->lock);
    WR_CUDA_TRY(cudaSetDevice(ctx->device));
    wr_cuda_model *m = new (std::nothrow) wr_cuda_model();
    if (!m) return WR_CUDA_ERR_NOMEM;
    m->ctx = ctx;
    m->n_layers = d->n_layers; m->hidden = d->hidden; m->n_q = d->n_q_heads; m->n_kv = d->n_kv_heads;
    m->hd = d->head_dim; m->vocab = d->vocab; m->n_rot = d->n_rot_pairs; m->max_rows = d->max_rows;
    m->eps = d->rms_eps; m->theta = d->rope_theta; m->scale = d->attn_scale;
    const size_t hid = d->hidden, nq = (size_t)d->n_q_heads * d->head_dim, nkv = (size_t)d->n_kv_heads * d->head_dim;
    const bool tied = (d->embed == d->lm_head);

    size_t total = up256((size_t)d->vocab * hid * 4) * (tied ? 1 : 2) + up256(hid * 4);
    for (uint32_t L = 0; L < d->n_layers; ++L) {
        const size_t ffn = d->layers[L].ffn_dim;
        if (ffn > m->ffn_max) m->ffn_max = (uint32_t)ffn;
        total += 2 * up256(hid * 4) + 2 * up256((size_t)d->head_dim * 4) + 2 * up256(nq * hid * 4) +
                 2 * up256(nkv * hid * 4) + 3 * up256(ffn * hid * 4);
    }
    const size_t R = d->max_rows, LR = kLogitRowsMax;
    const size_t scratch = up256(R * hid * 4) + 2 * up256(R * nq * 4) + 2 * up256(R * nkv * 4) +
                           up256(R * (size_t)m->ffn_max * 4) + up256(LR * hid * 4) +
                           up256(LR * (size_t)d->vocab * 4) + 2 * up256(R * 4) + 2 * up256(LR * kArgmaxParts * 4);
    m->slab_bytes = total + scratch;
    cudaError_t e = cudaMalloc(&m->slab, m->slab_bytes);
    if (e != cudaSuccess) {
        (void)cudaGetLastError();
        delete m;
        return WR_CUDA_ERR_NOMEM;
    }
    e = cudaHostAlloc((void **)&m->h_tokens, 2 * R * sizeof(uint32_t), cudaHostAllocPortable);
    if (e != cudaSuccess) {
        (void)cudaGetLastError();
        cudaFree(m->slab);
        delete m;
        return WR_CUDA_ERR_NOMEM;
    }
    char *cur = m->slab;
    bool ok = true;
    auto put = [&](const float *src, size_t n_floats) -> const float * {
        char *dst = cur;
        cur += up256(n_floats * 4);
        if (ok && cudaMemcpyAsync(dst, src, n_floats * 4, cudaMemcpyHostToDevice, ctx->stream) != cudaSuccess)
            ok = false;
        return reinterpret_cast<const float *>(dst);
    };
    auto take = [&](size_t n_floats) -> float * {
        char *dst = cur;
        cur += up256(n_floats * 4);
        return reinterpret_cast<float *>(dst);
    };
    m->lm_head = put(d->lm_head, (size_t)d->vocab * hid);
    m->embed = tied ? m->lm_head : put(d->embed, (size_t)d->vocab * hid);
    m->final_norm = put(d->final_norm, hid);
    m->layers.resize(d->n_layers);
    for (uint32_t L = 0; L < d->n_layers; ++L) {
        const wr_cuda_layer_desc &l = d->layers[L];
        wr_cuda_layer_dev &o = m->layers[L];
        const size_t ffn = l.ffn_dim;
        o.ffn = l.ffn_dim;
        o.attn_norm = put(l.attn_norm, hid);
        o.ffn_norm = put(l.ffn_norm, hid);
        o.q_norm = l.q_norm ? put(l.q_norm, d->head_dim) : nullptr;
        o.k_norm = l.k_norm ? put(l.k_norm, d->head_dim) : nullptr;
        if (!l.q_norm) cur += 2 * up256((size_t)d->head_dim * 4);
        o.wq = put(l.wq, nq * hid);
        o.wo = put(l.wo, nq * hid);
        o.wk = put(l.wk, nkv * hid);
        o.wv = put(l.wv, nkv * hid);
        o.w_gate = put(l.w_gate, ffn * hid);
        o.w_up = put(l.w_up, ffn * hid);
        o.w_down = put(l.w_down, ffn * hid);
    }
    m->resid = take(R * hid);
    m->q = take(R * nq);
    m->attn = take(R * nq);
    m->k = take(R * nkv);
    m->v = take(R * nkv);
    m->gate = take(R * (size_t)m->ffn_max);
    m->normed = take(LR * hid);
    m->logits = take(LR * (size_t)d->vocab);
    m->tokens = reinterpret_cast<uint32_t *>(take(R));
    m->best = reinterpret_cast<uint32_t *>(take(R));
    m->part_v = take(LR * kArgmaxParts);
    m->part_i = reinterpret_cast<uint32_t *>(take(LR * kArgmaxParts));
    if (ok && cudaStreamSynchronize(ctx->stream) != cudaSuccess) ok = false;
    if (!ok || (size_t)(cur - m->slab) > m->slab_bytes) {
        (void)cudaGetLastError();
        cudaFreeHost(m->h_tokens);
        cudaFree(m->slab);
        delete m;
        return WR_CUDA_ERR_INTERNAL;
    }
    *out = m;
    return WR_CUDA_OK;
}

extern "C" void wr_cuda_model_destroy(wr_cuda_model *m)
{
    if (!m) return;
    {
        std::lock_guard<std::mutex> g(m->ctx->lock);
        cudaSetDevice(m->ctx->device);
        cudaStreamSynchronize(m->ctx->stream);
        if (m->mixed) wr_mixed_destroy(m->mixed);
        cudaFree(m->slab);
        cudaFreeHost(m->h_tokens);
    }
    delete m;
}

extern "C" uint64_t wr_cuda_model_bytes(const wr_cuda_model *m) { return m ? m->slab_bytes : 0; }
extern "C" uint64_t wr_cuda_model_launches(const wr_cuda_model *m) { return m ? m->launches : 0; }
extern "C" uint64_t wr_cuda_model_last_enqueue_ns(const wr_cuda_model *m) { return m ? m->last_enqueue_ns : 0; }

extern "C" int wr_cuda_model_forward(wr_cuda_ctx *ctx, wr_cuda_model *m, int mode, uint32_t n_rows,
                                     wr_cuda_kv *const *kv, const uint32_t *positions,
                                     const uint32_t *tokens, uint32_t out_from, float *hidden_out,
                                     float *normed_out, float *const *logits_out, uint32_t *argmax_out,
                                     float *attn_tap_out)
{
    if (!ctx || !m || m->ctx != ctx || !kv || !positions || !tokens) return WR_CUDA_ERR_INVAL;
    if (mode != WR_CUDA_FWD_DECODE && mode != WR_CUDA_FWD_PREFILL) return WR_CUDA_ERR_INVAL;
    if (m->mixed) {
        if (attn_tap_out) return WR_CUDA_ERR_UNSUPPORTED;
        return wr_mixed_forward(ctx, m, mode, n_rows, kv, positions, tokens, out_from, hidden_out, normed_out,
                                logits_out, argmax_out);
    }
    if (n_rows == 0 || n_rows > m->max_rows || out_from > n_rows) return WR_CUDA_ERR_LIMIT;
    if (mode == WR_CUDA_FWD_DECODE && n_rows > WR_CUDA_BATCH_MAX) return WR_CUDA_ERR_LIMIT;
    const uint32_t n_out = n_rows - out_from;
    if ((logits_out || argmax_out) && n_out > kLogitRowsMax) return WR_CUDA_ERR_LIMIT;
    if ((normed_out || logits_out || argmax_out) && n_out == 0) return WR_CUDA_ERR_INVAL;
    for (uint32_t r = 0; r < n_rows; ++r)
        if (tokens[r] >= m->vocab) return WR_CUDA_ERR_INVAL;      // refused before anything runs
    const uint32_t n_sess = (mode == WR_CUDA_FWD_DECODE) ? n_rows : 1;
    for (uint32_t s = 0; s < n_sess; ++s)
        if (!kv[s] || kv[s]->n_layers != m->n_layers || kv[s]->n_kv_at(0) != m->n_kv || kv[s]->hd_at(0) != m->hd)
            return WR_CUDA_ERR_INVAL;

    std::lock_guard<std::mutex> fg(m->fwd);
    const auto t_begin = std::chrono::steady_clock::now();
    cudaStream_t st = ctx->stream;
    const uint32_t hid = m->hidden, nq = m->n_q * m->hd, nkv = m->n_kv * m->hd;

    // Decode rows are processed in an order of their own: the sessions that the one-kernel
    // short-context step covers first, the others after them, so that each kind is a contiguous
    // block of rows.  Which kind a session is depends on that session alone.  perm[i] = caller's row.
    uint32_t perm[WR_CUDA_BATCH_MAX], pos_p[WR_CUDA_BATCH_MAX], n_short = 0;
    wr_cuda_kv *kv_p[WR_CUDA_BATCH_MAX];
    bool permuted = false;
    if (mode == WR_CUDA_FWD_DECODE) {
        const bool use_small = (getenv("WR_CUDA_STEP_SMALL_OFF") == nullptr);
        uint32_t n = 0;
        for (int pass = 0; pass < 2; ++pass)
            for (uint32_t r = 0; r < n_rows; ++r) {
                const bool small = use_small && wr_step_small_covers(kv[r], m->n_q, positions[r]);
                if (small == (pass == 0)) perm[n++] = r;
            }
        for (uint32_t i = 0; i < n_rows; ++i) {
            if (perm[i] != i) permuted = true;
            kv_p[i] = kv[perm[i]];
            pos_p[i] = positions[perm[i]];
            if (use_small && wr_step_small_covers(kv_p[i], m->n_q, pos_p[i])) n_short = i + 1;
            if (pos_p[i] >= kv_p[i]->max_ctx) return WR_CUDA_ERR_CTX_FULL;
        }
    }
    {
        std::lock_guard<std::mutex> g(ctx->lock);
        WR_CUDA_TRY(cudaSetDevice(ctx->device));
        for (uint32_t r = 0; r < n_rows; ++r)
            m->h_tokens[r] = tokens[mode == WR_CUDA_FWD_DECODE ? perm[r] : r];
        WR_CUDA_TRY(cudaMemcpyAsync(m->tokens, m->h_tokens, n_rows * sizeof(uint32_t),
                                    cudaMemcpyHostToDevice, st));
        embed_rows_kernel<<<n_rows, 128, 0, st>>>(m->tokens, m->embed, m->resid, hid);
        ++m->launches;
        WR_CUDA_TRY(cudaGetLastError());
    }
    for (uint32_t L = 0; L < m->n_layers; ++L) {
        const wr_cuda_layer_dev &l = m->layers[L];
        int rc;
        {
            std::lock_guard<std::mutex> g(ctx->lock);
            GemvParams p{};
            p.seg[0] = {l.wq, m->q, nq, nq};
            p.seg[1] = {l.wk, m->k, nkv, nkv};
            p.seg[2] = {l.wv, m->v, nkv, nkv};
            p.n_seg = 3;
            p.x = m->resid; p.x_stride = hid; p.k = hid; p.rows = n_rows;
            p.norm_w = l.attn_norm; p.eps = m->eps;
            rc = gemv(m, p, nq + 2 * nkv);
            if (rc != WR_CUDA_OK) return rc;
            const uint32_t r_lo = (mode == WR_CUDA_FWD_DECODE) ? n_short : 0;    // rows of the three-kernel path
            if (l.q_norm && r_lo < n_rows) {
                const uint32_t n_a = (n_rows - r_lo) * m->n_q, n_b = (n_rows - r_lo) * m->n_kv;
                head_rmsnorm_kernel<<<(n_a + n_b + 3) / 4, 128, 0, st>>>(m->q + (size_t)r_lo * nq, l.q_norm, n_a,
                                                                       m->k + (size_t)r_lo * nkv, l.k_norm, n_b,
                                                                       m->hd, m->eps);
                ++m->launches;
                WR_CUDA_TRY(cudaGetLastError());
            }
            if (mode == WR_CUDA_FWD_DECODE && n_short) {
                rc = wr_step_small_launch(ctx, n_short, kv_p, L, pos_p, m->q, m->k, m->v, m->attn, m->n_q,
                                          m->theta, m->n_rot, l.q_norm, l.k_norm, m->eps, m->scale);
                if (rc != WR_CUDA_OK) return rc;
            }
        }
        if (mode == WR_CUDA_FWD_DECODE) {
            if (n_short < n_rows) {
                rc = wr_cuda_decode_step(ctx, n_rows - n_short, kv_p + n_short, L, pos_p + n_short,
                                         m->q + (size_t)n_short * nq, m->k + (size_t)n_short * nkv,
                                         m->v + (size_t)n_short * nkv, m->attn + (size_t)n_short * nq, m->n_q,
                                         m->theta, m->n_rot, WR_CUDA_APPEND_ROPE, m->scale, 0, WR_CUDA_MEM_DEVICE);
                if (rc != WR_CUDA_OK) return rc;
            }
        } else {
            rc = wr_cuda_kv_append(ctx, 1, kv, L, positions, n_rows, m->k, m->v, m->q, m->n_q, m->theta,
                                   m->n_rot, WR_CUDA_APPEND_ROPE, WR_CUDA_MEM_DEVICE);
            if (rc != WR_CUDA_OK) return rc;
            rc = wr_cuda_attn_prefill(ctx, kv[0], L, positions[0], n_rows, m->q, WR_CUDA_F32, m->attn,
                                      m->n_q, m->scale, 0, WR_CUDA_MEM_DEVICE);
            if (rc != WR_CUDA_OK) return rc;
        }
        {
            std::lock_guard<std::mutex> g(ctx->lock);
            if (attn_tap_out) {
                float *dst = attn_tap_out + (size_t)L * n_rows * nq;
                if (!permuted) {
                    WR_CUDA_TRY(cudaMemcpyAsync(dst, m->attn, (size_t)n_rows * nq * 4, cudaMemcpyDeviceToHost, st));
                } else {
                    for (uint32_t i = 0; i < n_rows; ++i)
                        WR_CUDA_TRY(cudaMemcpyAsync(dst + (size_t)perm[i] * nq, m->attn + (size_t)i * nq,
                                                    (size_t)nq * 4, cudaMemcpyDeviceToHost, st));
                }
            }
            GemvParams p{};
            p.seg[0] = {l.wo, m->resid, hid, hid};
            p.n_seg = 1;
            p.x = m->attn; p.x_stride = nq; p.k = nq; p.rows = n_rows;
            p.add = m->resid; p.add_stride = hid;
            rc = gemv(m, p, hid);
            if (rc != WR_CUDA_OK) return rc;

            GemvParams f{};
            f.seg[0] = {l.w_gate, m->gate, l.ffn, m->ffn_max};
            f.seg[1] = {l.w_up, nullptr, l.ffn, 0};
            f.n_seg = 2;
            f.swiglu = 1;
            f.x = m->resid; f.x_stride = hid; f.k = hid; f.rows = n_rows;
            f.norm_w = l.ffn_norm; f.eps = m->eps;
            rc = gemv(m, f, l.ffn);
            if (rc != WR_CUDA_OK) return rc;

            GemvParams dn{};
            dn.seg[0] = {l.w_down, m->resid, hid, hid};
            dn.n_seg = 1;
            dn.x = m->gate; dn.x_stride = m->ffn_max; dn.k = l.ffn; dn.rows = n_rows;
            dn.add = m->resid; dn.add_stride = hid;
            rc = gemv(m, dn, hid);
            if (rc != WR_CUDA_OK) return rc;
        }
    }
    std::lock_guard<std::mutex> g(ctx->lock);
    // Device rows [o_lo, n_rows) are finished (final norm, LM head); device row i is the caller's row
    // perm[i] when the decode rows were reordered, and then every row is finished and only the asked
    // ones are copied out.
    const uint32_t o_lo = permuted ? 0u : out_from, n_fin = n_rows - o_lo;
    auto caller_row = [&](uint32_t i) { return permuted ? perm[i] : i; };
    if ((logits_out || argmax_out) && n_fin > kLogitRowsMax) return WR_CUDA_ERR_LIMIT;
    const float *res_out = m->resid + (size_t)o_lo * hid;
    if (hidden_out && n_out) {
        if (!permuted) {
            WR_CUDA_TRY(cudaMemcpyAsync(hidden_out, res_out, (size_t)n_out * hid * 4, cudaMemcpyDeviceToHost, st));
        } else {
            for (uint32_t i = 0; i < n_rows; ++i)
                if (perm[i] >= out_from)
                    WR_CUDA_TRY(cudaMemcpyAsync(hidden_out + (size_t)(perm[i] - out_from) * hid,
                                                m->resid + (size_t)i * hid, (size_t)hid * 4,
                                                cudaMemcpyDeviceToHost, st));
        }
    }
    if ((normed_out || logits_out || argmax_out) && n_out) {
        // the final norm of at most 16 rows is kept for the LM head; more rows (normed_out only) go in passes
        for (uint32_t done = 0; done < n_fin; done += kLogitRowsMax) {
            const uint32_t nr = (n_fin - done < kLogitRowsMax) ? n_fin - done : kLogitRowsMax;
            rmsnorm_rows_kernel<<<nr, 256, 0, st>>>(res_out + (size_t)done * hid, hid, m->final_norm, m->normed,
                                                    hid, hid, m->eps);
            ++m->launches;
            WR_CUDA_TRY(cudaGetLastError());
            if (normed_out) {
                if (!permuted) {
                    WR_CUDA_TRY(cudaMemcpyAsync(normed_out + (size_t)done * hid, m->normed, (size_t)nr * hid * 4,
                                                cudaMemcpyDeviceToHost, st));
                } else {
                    for (uint32_t i = 0; i < nr; ++i)
                        if (perm[done + i] >= out_from)
                            WR_CUDA_TRY(cudaMemcpyAsync(normed_out + (size_t)(perm[done + i] - out_from) * hid,
                                                        m->normed + (size_t)i * hid, (size_t)hid * 4,
                                                        cudaMemcpyDeviceToHost, st));
                }
            }
        }
    }
    if ((logits_out || argmax_out) && n_out) {
        GemvParams p{};
        p.seg[0] = {m->lm_head, m->logits, m->vocab, m->vocab};
        p.n_seg = 1;
        p.x = m->normed; p.x_stride = hid; p.k = hid; p.rows = n_fin;
        int rc = gemv(m, p, m->vocab);
        if (rc != WR_CUDA_OK) return rc;
        if (argmax_out) {
            rc = wr_argmax_launch(st, m->logits, m->vocab, m->vocab, n_fin, m->part_v, m->part_i, m->best);
            if (rc != WR_CUDA_OK) return rc;
            m->launches += 2;
            WR_CUDA_TRY(cudaMemcpyAsync(m->h_tokens + m->max_rows, m->best, n_fin * sizeof(uint32_t),
                                        cudaMemcpyDeviceToHost, st));
        }
        if (logits_out)
            for (uint32_t i = 0; i < n_fin; ++i) {
                const uint32_t c = caller_row(o_lo + i);
                if (c >= out_from && logits_out[c - out_from])
                    WR_CUDA_TRY(cudaMemcpyAsync(logits_out[c - out_from], m->logits + (size_t)i * m->vocab,
                                                (size_t)m->vocab * 4, cudaMemcpyDeviceToHost, st));
            }
    }
    m->last_enqueue_ns = (uint64_t)std::chrono::duration_cast<std::chrono::nanoseconds>(
                             std::chrono::steady_clock::now() - t_begin).count();
    int rc = wr_ctx_sync_checked(ctx);
    if (rc != WR_CUDA_OK) return rc;
    if (argmax_out)
        for (uint32_t i = 0; i < n_fin; ++i) {
            const uint32_t c = caller_row(o_lo + i);
            if (c >= out_from) argmax_out[c - out_from] = m->h_tokens[m->max_rows + i];
        }
    return WR_CUDA_OK;
}
