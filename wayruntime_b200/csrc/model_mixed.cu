// model_mixed.cu — the layer stack of models whose layers differ (wr_cuda_model_create_mixed).
//
// The stack is a run list over layers; each layer is norm -> (token shift) -> mixer -> residual, then
// norm -> feed-forward -> residual, or (parallel) norm -> mixer + feed-forward -> residual.  An F32 model's projections are the products of gemv.cu.  A BF16 model's are
// tensor-core products: steps of up to WR_CUDA_BATCH_MAX rows (every decode step, and short portions of a prompt)
// keep F32 activations and take the weight-streaming one (gemm_skinny.cu), longer portions keep BF16 activations
// and take gemm_bf16.cu.  The residual stream, norms, softmax and recurrences are F32 in all of them.
//
// A session (wr_cuda_kv) holds K/V pages for the attention runs and two slots of recurrent state; a step reads
// the slot that stands at its first position and writes the other, so nothing a failed step does is kept.
#include <cuda_bf16.h>
#include <math.h>

#include <algorithm>
#include <chrono>
#include <cstring>
#include <new>

#include "gemm_bf16.cuh"
#include "gemv.cuh"
#include "mixers.cuh"
#include "model.cuh"

namespace {

constexpr uint32_t kHeadRows = 128;      // wanted rows finished (final norm, head) in one go
constexpr uint32_t kHd = 128;            // head_dim of the framework's F16 prefill / decode kernels
constexpr double kLog2e = 1.4426950408889634;

size_t up256(size_t n) { return (n + 255u) & ~(size_t)255u; }

constexpr uint32_t kMoeTile = 128;       // rows of a tile of gemm_bf16.cu

struct Mat {                             // [n][k]: F32 rows wr_ld(k) apart, or BF16 blocks (wr_weight)
    const void *w = nullptr;
    uint32_t n = 0, k = 0;
    CUtensorMap x_map{}, xs_map{};       // BF16 models: its input rows, and its input as split rows
    wr_pair_args pair;                   // BF16 models: gate and up rows side by side (where they lie, act)
};

struct Layer {
    uint32_t mixer = 0, ffn = WR_CUDA_FFN_NONE;
    const float *norm1 = nullptr, *norm2 = nullptr, *shift = nullptr;
    // attention
    wr_attn_geom g{};
    Mat qkvg, o;
    const float *qkv_bias = nullptr;
    uint32_t k_off = 0, v_off = 0, g_off = 0, proj_ld = 0;
    bool gated = false;
    uint32_t temp_every = 0;
    float temp_coef = 0.f, scale = 0.f, lambda = 0.f, diff_init = 0.f, diff_eps = 0.f;
    // selective scan
    uint32_t inner = 0, state = 0, rank = 0, taps = 0, b_off = 0, c_off = 0, dbc_ld = 0;
    Mat in, x, dt, out;
    const float *conv = nullptr, *conv_b = nullptr, *dt_b = nullptr, *a2 = nullptr, *d = nullptr;
    uint64_t conv_off = 0, scan_off = 0; // inside the run's state (token shift first)
    // feed-forward
    uint32_t ff = 0;
    Mat up, down;
    float act[4] = {0, 0, 0, 0}, ffn_eps = 0.f;
    // gated feed-forward: gate and up rows are part of `first` and its down columns part of `o` where a latent
    // layer's sublayers read one norm (fused); else products of their own.  F32: gate and `up` by themselves.
    bool parallel = false, fused = false;
    Mat gate;
    uint32_t ff_at = 0;                  // where the feed-forward's values lie in a row of `o`'s input (fused)
    // attention over a latent: `first` = [query latent | latent | rotated key part | router | gate and up]
    wr_latent_geom lat{};
    Mat first, uq;
    Mat ukv;                             // key rows of all heads, then value rows (BF16 models: F16 values)
    bool flash = false, tensor_decode = false;                   // prompts / few rows on the tensor cores
    const float *q_norm = nullptr, *c_norm = nullptr;
    const double *turns = nullptr;
    uint32_t rot_off = 0, logit_off = 0, kv_from = 0;
    float latent_eps = 0.f;
    // mixture of experts: gate and up of all experts, down of all experts
    uint32_t experts = 0, top = 0;
    float alpha = 0.f, limit = 0.f;
    Mat router, e_up, e_down;            // (n, k of one expert)
    size_t up_stride = 0, down_stride = 0;                       // bytes; F32: gate, then up_at floats behind it up
    size_t up_at = 0;
    const float *router_b = nullptr;
    wr_cuda_cache_layer cache{};
};

}  // namespace

struct wr_mixed {
    int compute = WR_CUDA_F32;
    uint32_t width = 0, ldw = 0, max_rows = 0, groups = 1;
    float eps = 0.f, embed_scale = 1.f, residual_mult = 1.f;
    bool centre = false;                 // layer norm
    std::vector<Layer> layers;
    std::vector<uint32_t> runs, rows_of; // rows_of: the run whose cache a run reads
    std::vector<uint64_t> state_off;     // per run, inside a session's slot
    std::vector<wr_cuda_cache_layer> cache;
    uint64_t state_bytes = 0;
    char *weights = nullptr;
    size_t weight_bytes = 0, scratch_bytes = 0;
    char *scratch = nullptr;
    const void *embed = nullptr;
    const double *turns = nullptr;       // sinusoidal position frequencies, or null
    const float *final_norm = nullptr;
    Mat head;
    // row scratch
    float *resid = nullptr, *dbc = nullptr, *dt = nullptr, *attn = nullptr, *logits = nullptr, *normed = nullptr;
    float *conv_f32 = nullptr;           // few rows of a BF16 model: the convolution for the scan (mid has it split)
    void *xin = nullptr, *proj = nullptr, *mid = nullptr, *scan_out = nullptr, *q = nullptr, *dbc16 = nullptr, *head_in = nullptr;
    // latent attention: first product's rows, query latent, queries in the latent, attended latents
    float *lat = nullptr, *qa = nullptr, *olat = nullptr;
    void *cq = nullptr;
    // experts: choice, places, gathered inputs, activations, results
    float *e_weight = nullptr;
    uint32_t *e_expert = nullptr, *e_place = nullptr, *e_row_of = nullptr, *e_list = nullptr, *e_count = nullptr;
    void *e_in = nullptr, *e_act = nullptr, *e_out = nullptr;
    uint32_t *tokens = nullptr, *gather = nullptr, *best = nullptr, *part_i = nullptr;
    float *part_v = nullptr;
    wr_seq_dev *seqs = nullptr;
    // pinned staging: tokens, gathered row numbers, session descriptors
    uint32_t *h_tokens = nullptr, *h_gather = nullptr, *h_best = nullptr;
    wr_seq_dev *h_seqs = nullptr;
    float *hidden_tap = nullptr;
};

namespace {

float bf16_to_f32(uint16_t b)
{
    uint32_t u = (uint32_t)b << 16;
    float f;
    memcpy(&f, &u, 4);
    return f;
}
uint16_t f32_to_bf16(float f)
{
    uint32_t u;
    memcpy(&u, &f, 4);
    if ((u & 0x7fffffffu) > 0x7f800000u) return (uint16_t)((u >> 16) | 0x40u);
    return (uint16_t)((u + 0x7fffu + ((u >> 16) & 1u)) >> 16);
}
uint16_t f32_to_f16(float f)
{
    const __half h = __float2half_rn(std::min(std::max(f, -65504.f), 65504.f));
    uint16_t u;
    memcpy(&u, &h, 2);
    return u;
}
float elem(const wr_cuda_tensor &t, size_t i)
{
    return t.dtype == WR_CUDA_BF16 ? bf16_to_f32(static_cast<const uint16_t *>(t.data)[i])
                                   : static_cast<const float *>(t.data)[i];
}

// Rows [row0, row0 + n) of a tensor at row `at` of a stacked weight, columns from `col` on.  Rows may come in groups that
// lie `stride` apart, the rows of a group from `first` on at `second`.
struct Part {
    const wr_cuda_tensor *t;
    uint32_t row0, n, at;
    uint32_t col = 0, k = 0;             // k: the tensor's row length where it is not the stacked weight's
    uint32_t group = ~0u, stride = 0, first = ~0u, second = 0;
    uint32_t dst(uint32_t r) const
    {
        const uint32_t w = r % group;
        return at + r / group * stride + (w < first ? w : second + w - first);
    }
    Part &in_groups(uint32_t g, uint32_t s, uint32_t f = ~0u, uint32_t f_at = 0)
    {
        group = g; stride = s; first = f; second = f_at;
        return *this;
    }
};
typedef std::vector<Part> Parts;

// Weights are laid out in host memory first (sizes are known once everything is placed), then copied in one go.
struct Packer {
    std::vector<uint8_t> buf;
    size_t at = 0;
    size_t place(size_t bytes)
    {
        const size_t o = at;
        at += up256(bytes);
        if (buf.size() < at) buf.resize(std::max(at, buf.size() * 2), 0);
        return o;
    }
    size_t floats(size_t n, size_t pad_to)
    {
        return place(std::max(n, pad_to) * 4);
    }
    float *f(size_t off) { return reinterpret_cast<float *>(buf.data() + off); }
    size_t vec(const wr_cuda_tensor &t, size_t n)
    {
        const size_t o = floats(n, wr_ld((uint32_t)n));
        for (size_t i = 0; i < n; ++i) f(o)[i] = elem(t, i);
        return o;
    }
    // [rows][k] out of parts, zeros elsewhere: rows wr_ld(k) apart in `type` ...
    size_t rows_of(const Parts &parts, uint32_t rows, uint32_t k, int type)
    {
        const size_t ld = wr_ld(k), es = type == WR_CUDA_BF16 ? 2 : 4;
        const size_t o = place(((size_t)rows * ld) * es);
        for (const Part &p : parts)
            for (uint32_t r = 0; r < p.n; ++r) {
                uint8_t *dst = buf.data() + o + ((size_t)p.dst(r) * ld + p.col) * es;
                const uint32_t pk = p.k ? p.k : k;
                const size_t src = (size_t)(p.row0 + r) * pk;
                for (uint32_t i = 0; i < pk; ++i) {
                    if (type == WR_CUDA_BF16) reinterpret_cast<uint16_t *>(dst)[i] = bits(*p.t, src + i);
                    else reinterpret_cast<float *>(dst)[i] = elem(*p.t, src + i);
                }
            }
        return o;
    }
    // ... or, for the products of a BF16 model, in blocks (wr_weight) of BF16 or F16 values
    size_t mat(const Parts &parts, uint32_t rows, uint32_t k, int type)
    {
        if (type == WR_CUDA_F32) return rows_of(parts, rows, k, type);
        const size_t o = place(wr_weight_bytes(rows, k));
        for (const Part &p : parts)
            for (uint32_t r = 0; r < p.n; ++r) {
                const uint32_t pk = p.k ? p.k : k;
                const size_t src = (size_t)(p.row0 + r) * pk;
                for (uint32_t i = 0; i < pk; i += 8) {           // pieces of eight stay together (col: a multiple of 8)
                    uint16_t *dst = reinterpret_cast<uint16_t *>(buf.data() + o + wr_weight_off(k, p.dst(r), p.col + i));
                    const uint32_t n = std::min(8u, pk - i);
                    if (type == WR_CUDA_F16)
                        for (uint32_t e = 0; e < n; ++e) dst[e] = f32_to_f16(elem(*p.t, src + i + e));
                    else if (p.t->dtype == WR_CUDA_BF16) memcpy(dst, static_cast<const uint16_t *>(p.t->data) + src + i, n * 2);
                    else
                        for (uint32_t e = 0; e < n; ++e) dst[e] = f32_to_bf16(elem(*p.t, src + i + e));
                }
            }
        return o;
    }
    static uint16_t bits(const wr_cuda_tensor &t, size_t i)
    {
        return t.dtype == WR_CUDA_BF16 ? static_cast<const uint16_t *>(t.data)[i] : f32_to_bf16(elem(t, i));
    }
};

bool has(const wr_cuda_tensor &t) { return t.data != nullptr; }
bool valid(const wr_cuda_tensor &t) { return !t.data || t.dtype == WR_CUDA_F32 || t.dtype == WR_CUDA_BF16; }

int check_layer(const wr_cuda_mixed_layer &l)
{
    for (const wr_cuda_tensor *t : {&l.norm1, &l.norm2, &l.shift, &l.wq, &l.wk, &l.wv, &l.wo, &l.bq, &l.bk, &l.bv, &l.w_gate,
                                    &l.lq1, &l.lk1, &l.lq2, &l.lk2, &l.w_in, &l.conv, &l.conv_b, &l.w_x, &l.w_dt, &l.dt_b,
                                    &l.a_log, &l.d, &l.w_out, &l.w_up, &l.w_down, &l.act, &l.w_dq, &l.dq_norm, &l.w_uq, &l.w_dkv,
                                    &l.dkv_norm, &l.w_uk, &l.w_uv, &l.w_gate_up, &l.router, &l.router_b})
        if (!valid(*t)) return WR_CUDA_ERR_INVAL;
    if (!has(l.norm1)) return WR_CUDA_ERR_INVAL;
    if (l.mixer == WR_CUDA_MIXER_ATTENTION) {
        if (!l.n_q_heads || !l.n_kv_heads || !l.k_dim || !l.v_dim || l.n_q_heads % l.n_kv_heads) return WR_CUDA_ERR_INVAL;
        if (l.n_maps != 1 && l.n_maps != 2) return WR_CUDA_ERR_UNSUPPORTED;
        if (!has(l.wq) || !has(l.wk) || !has(l.wv) || !has(l.wo)) return WR_CUDA_ERR_INVAL;
        if (l.n_maps == 2 && (!has(l.lq1) || !has(l.lk1) || !has(l.lq2) || !has(l.lk2))) return WR_CUDA_ERR_INVAL;
        if (l.v_dim > 512 || l.n_maps * l.k_dim > WR_CUDA_HEAD_DIM_MAX) return WR_CUDA_ERR_LIMIT;
    } else if (l.mixer == WR_CUDA_MIXER_MAMBA1) {
        if (!l.inner || !l.state || !l.dt_rank || !l.taps) return WR_CUDA_ERR_INVAL;
        if (!has(l.w_in) || !has(l.conv) || !has(l.w_x) || !has(l.w_dt) || !has(l.a_log) || !has(l.d) || !has(l.w_out))
            return WR_CUDA_ERR_INVAL;
        if (l.state > 512) return WR_CUDA_ERR_LIMIT;
    } else if (l.mixer == WR_CUDA_MIXER_LATENT) {
        if (!l.n_q_heads || !l.k_dim || !l.v_dim || !l.rot_dim || l.rot_dim % 2 || !l.q_rank || !l.kv_rank || !(l.rope_base > 0))
            return WR_CUDA_ERR_INVAL;
        if (!has(l.w_dq) || !has(l.dq_norm) || !has(l.w_uq) || !has(l.w_uk) || !has(l.w_uv) || !has(l.wo)) return WR_CUDA_ERR_INVAL;
        if (!l.kv_from && (!has(l.w_dkv) || !has(l.dkv_norm))) return WR_CUDA_ERR_INVAL;
        if (l.kv_rank > 512 || l.rot_dim > 256 || l.k_dim > WR_CUDA_HEAD_DIM_MAX || l.v_dim > WR_CUDA_HEAD_DIM_MAX)
            return WR_CUDA_ERR_LIMIT;
    } else {
        return WR_CUDA_ERR_UNSUPPORTED;
    }
    if (l.ffn != WR_CUDA_FFN_NONE && !l.parallel && !has(l.norm2)) return WR_CUDA_ERR_INVAL;
    if (l.parallel && l.mixer != WR_CUDA_MIXER_LATENT && has(l.shift)) return WR_CUDA_ERR_UNSUPPORTED;
    if (l.ffn == WR_CUDA_FFN_SWIGLU) {
        if (!l.ffn_dim || !has(l.w_gate_up) || !has(l.w_up) || !has(l.w_down)) return WR_CUDA_ERR_INVAL;
    } else if (l.ffn == WR_CUDA_FFN_MOE) {
        if (!l.ffn_dim || !l.n_experts || !l.top_k || l.top_k > l.n_experts || !has(l.router) || !has(l.router_b) || !l.experts)
            return WR_CUDA_ERR_INVAL;
        if (l.n_experts > 2048) return WR_CUDA_ERR_LIMIT;
        for (uint32_t i = 0; i < 3 * l.n_experts; ++i)
            if (!has(l.experts[i]) || !valid(l.experts[i])) return WR_CUDA_ERR_INVAL;
    } else if (l.ffn == WR_CUDA_FFN_POLYNORM) {
        if (!l.ffn_dim || !has(l.w_up) || !has(l.w_down) || !has(l.act)) return WR_CUDA_ERR_INVAL;
    } else if (l.ffn != WR_CUDA_FFN_NONE) {
        return WR_CUDA_ERR_UNSUPPORTED;
    }
    return WR_CUDA_OK;
}

double dot_exp(const wr_cuda_tensor &a, const wr_cuda_tensor &b, uint32_t n)
{
    double s = 0;
    for (uint32_t i = 0; i < n; ++i) s += (double)elem(a, i) * (double)elem(b, i);
    return exp(s);
}

// Everything about a layer that needs no device memory yet: weight offsets are kept where the pointers go later.
template <typename P> void set_off(P *&p, size_t off) { p = reinterpret_cast<P *>(off + 1); }    // (0 stays "absent")

void pack_layer(Packer &pk, const wr_cuda_mixed_layer &l, Layer &o, uint32_t width, int type)
{
    auto mat = [&](Mat &m, const Parts &parts, uint32_t n, uint32_t k) {
        m.n = n;
        m.k = k;
        set_off(m.w, pk.mat(parts, n, k, type));
    };
    const bool bf = type == WR_CUDA_BF16;
    o.mixer = l.mixer;
    o.ffn = l.ffn;
    o.parallel = l.parallel != 0;
    o.fused = o.parallel && l.mixer == WR_CUDA_MIXER_LATENT && l.ffn == WR_CUDA_FFN_SWIGLU;
    o.ff = l.ffn == WR_CUDA_FFN_NONE ? 0 : l.ffn_dim;
    // gate and up rows from row `at` of a weight on, eight of one and eight of the other
    auto pairs = [&](Parts &p, const wr_cuda_tensor &gate, const wr_cuda_tensor &up, uint32_t at) {
        p.push_back(Part{&gate, 0, l.ffn_dim, at}.in_groups(8, 16));
        p.push_back(Part{&up, 0, l.ffn_dim, at + 8}.in_groups(8, 16));
    };
    const uint32_t pair_rows = 2 * wr_ld(l.ffn_dim);
    set_off(o.norm1, pk.vec(l.norm1, width));
    if (has(l.shift)) {
        set_off(o.shift, pk.vec(l.shift, width));
        o.cache.state_bytes = up256((size_t)width * 4);
    }
    if (l.mixer == WR_CUDA_MIXER_ATTENTION) {
        wr_attn_geom &g = o.g;
        g.n_q = l.n_q_heads; g.n_kv = l.n_kv_heads; g.maps = l.n_maps; g.kd = l.k_dim; g.vd = l.v_dim;
        const uint32_t kw = g.maps * g.kd;
        g.hd128 = type == WR_CUDA_BF16 && kw <= kHd && g.vd <= kHd;
        if (g.hd128) g.kv = {g.n_kv, kHd, kHd, WR_CUDA_F16};
        else g.kv = {g.n_kv, kw, g.vd, type == WR_CUDA_BF16 ? (uint32_t)WR_CUDA_F16 : (uint32_t)WR_CUDA_F32};
        o.cache.n_kv_heads = g.kv.n_kv; o.cache.k_dim = g.kv.k_dim; o.cache.v_dim = g.kv.v_dim; o.cache.elem = g.kv.elem;
        const uint32_t nq = g.n_q * kw, nk = g.n_kv * kw, nv = g.n_kv * g.vd, ng = g.n_q * g.vd;
        o.gated = has(l.w_gate);
        o.k_off = wr_ld(nq);
        o.v_off = o.k_off + wr_ld(nk);
        o.g_off = o.v_off + wr_ld(nv);
        const uint32_t n = o.gated ? o.g_off + ng : o.v_off + nv;
        o.proj_ld = wr_ld(n);
        mat(o.qkvg, {{&l.wq, 0, nq, 0}, {&l.wk, 0, nk, o.k_off}, {&l.wv, 0, nv, o.v_off},
                     {&l.w_gate, 0, o.gated ? ng : 0u, o.g_off}}, n, width);
        if (has(l.bq) || has(l.bk) || has(l.bv)) {
            const size_t b = pk.floats(n, o.proj_ld);
            for (uint32_t i = 0; i < nq && has(l.bq); ++i) pk.f(b)[i] = elem(l.bq, i);
            for (uint32_t i = 0; i < nk && has(l.bk); ++i) pk.f(b)[o.k_off + i] = elem(l.bk, i);
            for (uint32_t i = 0; i < nv && has(l.bv); ++i) pk.f(b)[o.v_off + i] = elem(l.bv, i);
            set_off(o.qkv_bias, b);
        }
        mat(o.o, {{&l.wo, 0, width, 0}}, width, ng);
        o.temp_every = l.q_temp_every;
        o.temp_coef = l.q_temp_coef;
        o.scale = l.attn_scale;
        o.diff_init = l.diff_init;
        o.diff_eps = l.diff_eps;
        if (g.maps == 2)
            o.lambda = (float)(dot_exp(l.lq1, l.lk1, g.kd) - dot_exp(l.lq2, l.lk2, g.kd) + (double)l.diff_init);
    } else if (l.mixer == WR_CUDA_MIXER_LATENT) {
        wr_latent_geom &g = o.lat;
        g = {l.n_q_heads, l.k_dim, l.rot_dim, l.v_dim, l.q_rank, l.kv_rank};
        o.kv_from = l.kv_from;
        o.latent_eps = l.latent_eps;
        o.scale = l.attn_scale;
        o.g.n_q = g.heads; o.g.n_kv = 1; o.g.maps = 1; o.g.kd = g.row(); o.g.vd = g.kv_rank; o.g.shared = true;
        o.g.kv = {1, g.row(), 0, bf ? (uint32_t)WR_CUDA_F16 : (uint32_t)WR_CUDA_F32};
        if (!l.kv_from) { o.cache.n_kv_heads = 1; o.cache.k_dim = g.row(); o.cache.elem = o.g.kv.elem; }
        const bool moe = o.parallel && l.ffn == WR_CUDA_FFN_MOE;
        Parts p = {{&l.w_dq, 0, g.q_rank, 0}};
        uint32_t n = wr_ld(g.q_rank);
        if (!l.kv_from) {
            o.k_off = n;
            o.rot_off = o.k_off + wr_ld(g.kv_rank);
            n = o.rot_off + wr_ld(g.rot);
            p.push_back({&l.w_dkv, 0, g.kv_rank, o.k_off});
            p.push_back({&l.w_dkv, g.kv_rank, g.rot, o.rot_off});
        }
        if (moe) {
            o.logit_off = n;
            n += wr_ld(l.n_experts);
            p.push_back({&l.router, 0, l.n_experts, o.logit_off});
        }
        if (o.fused && bf) n = (n + 15u) & ~15u;
        o.proj_ld = n;                                   // (the plain rows' outputs, zeros up to the first pair included)
        if (o.fused && bf) {
            o.first.pair.from = n;
            pairs(p, l.w_gate_up, l.w_up, n);
            n += pair_rows;
        }
        mat(o.first, p, n, width);
        mat(o.uq, {Part{&l.w_uq, 0, g.heads * (g.dim + g.rot), 0}.in_groups(g.dim + g.rot, g.q_head(), g.dim, g.dim_pad())},
            g.heads * g.q_head(), g.q_rank);
        const int half = bf ? WR_CUDA_F16 : WR_CUDA_F32;
        o.ukv.n = g.heads * (g.dim_pad() + g.vdim_pad());
        o.ukv.k = g.kv_rank;
        set_off(o.ukv.w, pk.mat({Part{&l.w_uk, 0, g.heads * g.dim, 0}.in_groups(g.dim, g.dim_pad()),
                                 Part{&l.w_uv, 0, g.heads * g.vdim, g.heads * g.dim_pad()}.in_groups(g.vdim, g.vdim_pad())},
                                o.ukv.n, g.kv_rank, half));
        o.flash = bf && wr_latent_flash_covers(g, l.attn_scale);
        o.tensor_decode = bf && wr_latent_decode_covers(g);
        const uint32_t nv = g.heads * g.vdim;
        if (o.fused) {
            o.ff_at = wr_ld(nv);
            Part a{&l.wo, 0, width, 0}, b{&l.w_down, 0, width, 0};
            a.k = nv;
            b.k = l.ffn_dim;
            b.col = o.ff_at;
            mat(o.o, {a, b}, width, o.ff_at + l.ffn_dim);
        } else {
            mat(o.o, {{&l.wo, 0, width, 0}}, width, nv);
        }
        set_off(o.q_norm, pk.vec(l.dq_norm, g.q_rank));
        if (!l.kv_from) set_off(o.c_norm, pk.vec(l.dkv_norm, g.kv_rank));
        const size_t t = pk.place((size_t)g.rot / 2 * 8);
        for (uint32_t i = 0; i < g.rot / 2; ++i)
            reinterpret_cast<double *>(pk.buf.data() + t)[i] = pow(l.rope_base, -2.0 * i / g.rot) / 6.283185307179586476925;
        set_off(o.turns, t);
    } else {
        o.inner = l.inner; o.state = l.state; o.rank = l.dt_rank; o.taps = l.taps;
        const uint32_t ldi = wr_ld(l.inner), lds = wr_ld(l.state);
        o.b_off = wr_ld(l.dt_rank);
        o.c_off = o.b_off + lds;
        o.dbc_ld = o.c_off + lds;
        // x at 0 and z at ldi; dt, B and C on boundaries of eight
        mat(o.in, {{&l.w_in, 0, l.inner, 0}, {&l.w_in, l.inner, l.inner, ldi}}, 2 * ldi, width);
        mat(o.x, {{&l.w_x, 0, l.dt_rank, 0}, {&l.w_x, l.dt_rank, l.state, o.b_off},
                  {&l.w_x, l.dt_rank + l.state, l.state, o.c_off}}, o.dbc_ld, l.inner);
        mat(o.dt, {{&l.w_dt, 0, l.inner, 0}}, l.inner, l.dt_rank);
        mat(o.out, {{&l.w_out, 0, width, 0}}, width, l.inner);
        const size_t cw = pk.floats((size_t)l.taps * ldi, 0);
        for (uint32_t c = 0; c < l.inner; ++c)
            for (uint32_t j = 0; j < l.taps; ++j) pk.f(cw)[(size_t)j * ldi + c] = elem(l.conv, (size_t)c * l.taps + j);
        set_off(o.conv, cw);
        const size_t cb = pk.floats(l.inner, ldi), db = pk.floats(l.inner, ldi);
        for (uint32_t c = 0; c < l.inner; ++c) {
            if (has(l.conv_b)) pk.f(cb)[c] = elem(l.conv_b, c);
            if (has(l.dt_b)) pk.f(db)[c] = elem(l.dt_b, c);
        }
        set_off(o.conv_b, cb);
        set_off(o.dt_b, db);
        const size_t a = pk.floats((size_t)l.inner * lds, 0);
        for (uint32_t c = 0; c < l.inner; ++c)
            for (uint32_t n = 0; n < l.state; ++n)
                pk.f(a)[(size_t)c * lds + n] = (float)(-exp((double)elem(l.a_log, (size_t)c * l.state + n)) * kLog2e);
        set_off(o.a2, a);
        set_off(o.d, pk.vec(l.d, l.inner));
        o.conv_off = o.cache.state_bytes;
        o.scan_off = o.conv_off + up256((size_t)(l.taps - 1) * ldi * 4);
        o.cache.state_bytes = o.scan_off + up256((size_t)l.inner * l.state * 4);
    }
    if (l.ffn == WR_CUDA_FFN_NONE) return;
    if (!o.parallel) set_off(o.norm2, pk.vec(l.norm2, width));
    if (l.ffn == WR_CUDA_FFN_POLYNORM) {
        o.ffn_eps = l.ffn_eps;
        mat(o.up, {{&l.w_up, 0, l.ffn_dim, 0}}, l.ffn_dim, width);
        mat(o.down, {{&l.w_down, 0, width, 0}}, width, l.ffn_dim);
        for (int i = 0; i < 4; ++i) o.act[i] = elem(l.act, i);
    } else if (l.ffn == WR_CUDA_FFN_SWIGLU) {
        if (!bf) {
            mat(o.gate, {{&l.w_gate_up, 0, l.ffn_dim, 0}}, l.ffn_dim, width);
            mat(o.up, {{&l.w_up, 0, l.ffn_dim, 0}}, l.ffn_dim, width);
        } else if (!o.fused) {
            Parts p;
            pairs(p, l.w_gate_up, l.w_up, 0);
            o.gate.pair.from = 0;
            mat(o.gate, p, pair_rows, width);
        }
        if (!o.fused) mat(o.down, {{&l.w_down, 0, width, 0}}, width, l.ffn_dim);
    } else {
        o.experts = l.n_experts; o.top = l.top_k; o.alpha = l.moe_alpha; o.limit = l.moe_limit;
        set_off(o.router_b, pk.vec(l.router_b, l.n_experts));
        if (!(o.parallel && l.mixer == WR_CUDA_MIXER_LATENT)) mat(o.router, {{&l.router, 0, l.n_experts, 0}}, l.n_experts, width);
        // expert after expert: every one takes a multiple of 256 bytes, so they lie one stride apart
        for (uint32_t e = 0; e < l.n_experts; ++e) {
            Parts p;
            if (bf) pairs(p, l.experts[3 * e], l.experts[3 * e + 1], 0);
            else p = {{&l.experts[3 * e], 0, l.ffn_dim, 0}, {&l.experts[3 * e + 1], 0, l.ffn_dim, l.ffn_dim}};
            const size_t at = pk.mat(p, bf ? pair_rows : 2 * l.ffn_dim, width, type);
            if (e == 0) set_off(o.e_up.w, at);
            if (e == 1) o.up_stride = at - (reinterpret_cast<size_t>(o.e_up.w) - 1);
        }
        for (uint32_t e = 0; e < l.n_experts; ++e) {
            const size_t at = pk.mat({{&l.experts[3 * e + 2], 0, width, 0}}, width, l.ffn_dim, type);
            if (e == 0) set_off(o.e_down.w, at);
            if (e == 1) o.down_stride = at - (reinterpret_cast<size_t>(o.e_down.w) - 1);
        }
        o.e_up.n = bf ? pair_rows : l.ffn_dim;
        o.e_up.k = width;
        o.up_at = (size_t)l.ffn_dim * wr_ld(width);
        o.e_up.pair.from = 0;
        o.e_up.pair.act = WR_PAIR_LIMITED;
        o.e_up.pair.alpha = l.moe_alpha;
        o.e_up.pair.limit = l.moe_limit;
        o.e_down.n = width;
        o.e_down.k = l.ffn_dim;
    }
}

template <typename P> void fix(P *&p, const char *base)
{
    if (p) p = reinterpret_cast<P *>(const_cast<char *>(base) + (reinterpret_cast<size_t>(p) - 1));
}

int fix_mat(Mat &m, const wr_mixed &x, const void *input, uint32_t input_rows, uint32_t input_ld, const void *few_input = nullptr,
            uint32_t groups = 1)
{
    if (!m.w) return WR_CUDA_OK;
    fix(m.w, x.weights);
    if (x.compute != WR_CUDA_BF16) return WR_CUDA_OK;
    int rc = wr_gemm_map_rows(&m.x_map, input, input_rows, m.k, input_ld);
    if (rc == WR_CUDA_OK) rc = wr_skinny_map_rows(&m.xs_map, few_input ? few_input : input, m.k, input_ld, groups);
    return rc;
}

}  // namespace

void wr_mixed_destroy(wr_mixed *x)
{
    if (!x) return;
    if (x->weights) (void)cudaFree(x->weights);
    if (x->scratch) (void)cudaFree(x->scratch);
    if (x->h_tokens) (void)cudaFreeHost(x->h_tokens);
    (void)cudaGetLastError();
    delete x;
}

extern "C" int wr_cuda_model_create_mixed(wr_cuda_ctx *ctx, const wr_cuda_mixed_desc *d, wr_cuda_model **out)
{
    if (!ctx || !d || !out) return WR_CUDA_ERR_INVAL;
    *out = nullptr;
    if (!d->width || !d->vocab || !d->n_layers || !d->layers || !d->n_runs || !d->runs || !d->max_rows || !d->norm_groups ||
        !has(d->embed) || !has(d->head) || !has(d->final_norm) || !valid(d->embed) || !valid(d->head) || !valid(d->final_norm))
        return WR_CUDA_ERR_INVAL;
    if (d->compute != WR_CUDA_F32 && d->compute != WR_CUDA_BF16) return WR_CUDA_ERR_INVAL;
    if (d->width % d->norm_groups) return WR_CUDA_ERR_INVAL;
    if (d->norm != WR_CUDA_NORM_RMS && d->norm != WR_CUDA_NORM_LAYER) return WR_CUDA_ERR_UNSUPPORTED;
    if (d->position != WR_CUDA_POS_NONE && d->position != WR_CUDA_POS_SINUSOIDAL) return WR_CUDA_ERR_UNSUPPORTED;
    if (d->n_runs > WR_CUDA_MAX_LAYER_RUNS) return WR_CUDA_ERR_LIMIT;
    for (uint32_t i = 0; i < d->n_runs; ++i)
        if (d->runs[i] >= d->n_layers) return WR_CUDA_ERR_INVAL;
    for (uint32_t L = 0; L < d->n_layers; ++L) {
        const int rc = check_layer(d->layers[L]);
        if (rc != WR_CUDA_OK) return rc;
    }
    // a run that borrows reads the latest earlier run of the named layer, whose rows must be laid out like its own
    std::vector<uint32_t> rows_of(d->n_runs);
    for (uint32_t i = 0; i < d->n_runs; ++i) {
        const wr_cuda_mixed_layer &l = d->layers[d->runs[i]];
        rows_of[i] = i;
        if (l.mixer != WR_CUDA_MIXER_LATENT || !l.kv_from) continue;
        uint32_t r = i;
        while (r > 0 && d->runs[r - 1] != l.kv_from - 1) --r;
        if (r == 0) return WR_CUDA_ERR_INVAL;
        const wr_cuda_mixed_layer &from = d->layers[l.kv_from - 1];
        if (from.mixer != WR_CUDA_MIXER_LATENT || from.kv_from || from.kv_rank != l.kv_rank || from.rot_dim != l.rot_dim ||
            from.rope_base != l.rope_base)
            return WR_CUDA_ERR_INVAL;
        rows_of[i] = r - 1;
    }
    std::lock_guard<std::mutex> g(ctx->lock);
    WR_CUDA_TRY(cudaSetDevice(ctx->device));
    wr_cuda_model *m = new (std::nothrow) wr_cuda_model();
    wr_mixed *x = new (std::nothrow) wr_mixed();
    if (!m || !x) {
        delete m;
        delete x;
        return WR_CUDA_ERR_NOMEM;
    }
    m->ctx = ctx;
    m->mixed = x;
    m->vocab = d->vocab;
    m->max_rows = d->max_rows;
    m->n_layers = d->n_runs;
    m->hidden = d->width;
    const int type = x->compute = (int)d->compute;
    const bool bf = type == WR_CUDA_BF16;
    x->width = d->width;
    x->ldw = wr_ld(d->width);
    x->max_rows = d->max_rows;
    x->groups = d->norm_groups;
    x->eps = d->norm_eps;
    x->centre = d->norm == WR_CUDA_NORM_LAYER;
    x->embed_scale = d->embed_scale;
    x->residual_mult = d->residual_mult;
    x->rows_of = rows_of;
    x->runs.assign(d->runs, d->runs + d->n_runs);

    Packer pk;
    set_off(x->embed, pk.rows_of({{&d->embed, 0, d->vocab, 0}}, d->vocab, d->width, type));
    x->head.n = d->vocab;
    x->head.k = d->width;
    set_off(x->head.w, pk.mat({{&d->head, 0, d->vocab, 0}}, d->vocab, d->width, type));
    set_off(x->final_norm, pk.vec(d->final_norm, d->width));
    if (d->position == WR_CUDA_POS_SINUSOIDAL) {
        const uint32_t pairs = (d->width + 1) / 2;
        const size_t o = pk.place((size_t)pairs * 8);
        for (uint32_t i = 0; i < pairs; ++i)
            reinterpret_cast<double *>(pk.buf.data() + o)[i] =
                pow((double)d->position_base, -2.0 * i / d->width) / 6.283185307179586476925;
        set_off(x->turns, o);
    }
    x->layers.resize(d->n_layers);
    for (uint32_t L = 0; L < d->n_layers; ++L) pack_layer(pk, d->layers[L], x->layers[L], d->width, type);
    for (uint32_t i = 0; i < d->n_runs; ++i) {
        const wr_cuda_cache_layer &c = x->layers[x->runs[i]].cache;
        x->cache.push_back(c);
        x->state_off.push_back(x->state_bytes);
        x->state_bytes += up256(c.state_bytes);      // as wr_cuda_kv_create_layout lays the slot out
    }
    x->weight_bytes = pk.at;

    // row scratch: what a step of few rows keeps in F32, a BF16 model's long step keeps in 16 bits
    const size_t R = std::max<uint32_t>(d->max_rows, WR_CUDA_BATCH_MAX), few = WR_CUDA_BATCH_MAX;
    size_t proj = 0, mid = x->ldw, q = 0, q_few = 0, att = 0, dbc = 0, scan = 0;
    size_t lat = 0, cq = 0, qa = 0, olat = 0, e_top = 0, e_list = 0, e_rows = 0, e_in = 0, e_act = 0, e_out = 0;
    for (const Layer &l : x->layers) {
        if (l.mixer == WR_CUDA_MIXER_ATTENTION) {
            proj = std::max<size_t>(proj, l.proj_ld);
            mid = std::max<size_t>(mid, wr_ld(l.g.n_q * l.g.vd));
            const size_t ql = (size_t)l.g.vq() * l.g.q_stride();
            q_few = std::max(q_few, ql);
            q = std::max(q, l.g.hd128 ? ql * 2 : ql * 4);
            att = std::max<size_t>(att, (size_t)l.g.vq() * l.g.o_stride());
        } else if (l.mixer == WR_CUDA_MIXER_LATENT) {
            const wr_latent_geom &g = l.lat;
            lat = std::max<size_t>(lat, l.proj_ld);
            cq = std::max<size_t>(cq, wr_ld(g.q_rank));
            q_few = std::max<size_t>(q_few, g.heads * g.q_head());
            q = std::max<size_t>(q, (size_t)g.heads * g.q_head() * 4);
            mid = std::max<size_t>(mid, wr_ld(l.o.k));
            const size_t n = l.flash ? few : R;          // rows that attend in the latent
            qa = std::max<size_t>(qa, std::max<size_t>(n * g.heads * g.row(), few * wr_latent_split_bytes(g) / 4));
            olat = std::max<size_t>(olat, n * g.heads * g.rank_pad());
        } else {
            proj = std::max<size_t>(proj, 2 * wr_ld(l.inner));
            mid = std::max<size_t>(mid, wr_ld(l.inner));
            dbc = std::max<size_t>(dbc, l.dbc_ld);
            scan = std::max<size_t>(scan, wr_ld(l.inner));
        }
        if (l.experts) {
            const uint32_t tile = bf ? kMoeTile : kMoeTileF32, tiles = wr_route_tiles((uint32_t)R, l.experts, l.top, tile);
            const size_t places = (size_t)tiles * tile, groups = wr_route_tiles((uint32_t)few, l.experts, l.top, 0);
            const size_t es = bf ? 2 : 4, lf = wr_ld(l.ff);
            lat = std::max<size_t>(lat, wr_ld(l.experts));
            e_top = std::max<size_t>(e_top, l.top);
            e_list = std::max<size_t>(e_list, std::max<size_t>(tiles, groups));
            e_rows = std::max<size_t>(e_rows, places);
            if (bf) e_in = std::max<size_t>(e_in, places * x->ldw * 2);
            e_act = std::max<size_t>(e_act, std::max(places * lf * es, bf ? groups * 2 * few * lf * 2 : 0));
            e_out = std::max<size_t>(e_out, std::max(places * x->ldw * es, bf ? groups * few * x->ldw * 4 : 0));
        } else if (l.ff) {
            proj = std::max<size_t>(proj, wr_ld(l.ff));
            mid = std::max<size_t>(mid, wr_ld(l.ff));
        }
    }
    auto act = [&](size_t per_row) { return bf ? std::max(R * per_row * 2, few * per_row * 4) : R * per_row * 4; };
    const size_t ldv = wr_ld(d->vocab);
    struct { void **p; size_t bytes; } want[] = {
        {(void **)&x->resid, R * x->ldw * 4}, {&x->xin, act(x->ldw)}, {&x->proj, act(proj)},
        {&x->mid, act(mid)}, {&x->scan_out, act(scan)}, {&x->q, std::max(R * q, few * q_few * 4)}, {(void **)&x->attn, R * att * 4},
        {(void **)&x->dbc, R * dbc * 4}, {&x->dbc16, bf ? std::max(R, 2 * few) * dbc * 2 : 0},
        {(void **)&x->lat, R * lat * 4}, {&x->cq, act(cq)}, {(void **)&x->qa, qa * 4}, {(void **)&x->olat, olat * 4},
        {(void **)&x->e_weight, R * e_top * 4}, {(void **)&x->e_expert, R * e_top * 4}, {(void **)&x->e_place, R * e_top * 4},
        {(void **)&x->e_row_of, e_rows * 4}, {(void **)&x->e_list, e_list * 4}, {(void **)&x->e_count, 4},
        {&x->e_in, e_in}, {&x->e_act, e_act}, {&x->e_out, e_out},
        {(void **)&x->conv_f32, bf ? few * scan * 4 : 0}, {(void **)&x->dt, R * scan * 4},
        {&x->head_in, (size_t)kHeadRows * x->ldw * 4}, {(void **)&x->normed, (size_t)kHeadRows * x->ldw * 4},
        {(void **)&x->logits, (size_t)kHeadRows * ldv * 4}, {(void **)&x->tokens, R * 4}, {(void **)&x->gather, R * 4},
        {(void **)&x->best, few * 4}, {(void **)&x->part_v, few * WR_ARGMAX_PARTS * 4},
        {(void **)&x->part_i, few * WR_ARGMAX_PARTS * 4}, {(void **)&x->seqs, few * sizeof(wr_seq_dev)},
    };
    for (auto &w : want) x->scratch_bytes += up256(w.bytes) + 256;
    auto fail = [&](int rc) {
        (void)cudaGetLastError();
        wr_mixed_destroy(x);
        delete m;
        return rc;
    };
    if (cudaMalloc((void **)&x->weights, x->weight_bytes) != cudaSuccess) return fail(WR_CUDA_ERR_NOMEM);
    if (cudaMalloc((void **)&x->scratch, x->scratch_bytes) != cudaSuccess) return fail(WR_CUDA_ERR_NOMEM);
    const size_t host_bytes = 2 * R * 4 + few * 4 + few * sizeof(wr_seq_dev) + 64;
    if (cudaHostAlloc((void **)&x->h_tokens, host_bytes, cudaHostAllocPortable) != cudaSuccess)
        return fail(WR_CUDA_ERR_NOMEM);
    x->h_gather = x->h_tokens + R;
    x->h_best = x->h_gather + R;
    x->h_seqs = reinterpret_cast<wr_seq_dev *>((reinterpret_cast<uintptr_t>(x->h_best + few) + 15u) & ~(uintptr_t)15u);
    // zeros first: pad columns that no kernel writes must hold finite values
    if (cudaMemsetAsync(x->scratch, 0, x->scratch_bytes, ctx->stream) != cudaSuccess ||
        cudaMemcpyAsync(x->weights, pk.buf.data(), x->weight_bytes, cudaMemcpyHostToDevice, ctx->stream) != cudaSuccess ||
        cudaStreamSynchronize(ctx->stream) != cudaSuccess)
        return fail(WR_CUDA_ERR_INTERNAL);
    char *cur = x->scratch;
    for (auto &w : want) {
        *w.p = cur;
        cur += up256(w.bytes) + 256;
    }
    m->slab_bytes = x->weight_bytes + x->scratch_bytes;

    fix(x->embed, x->weights);
    fix(x->turns, x->weights);
    fix(x->final_norm, x->weights);
    const uint32_t rows = (uint32_t)R;
    int rc = fix_mat(x->head, *x, x->head_in, kHeadRows, x->ldw);
    for (Layer &l : x->layers) {
        fix(l.norm1, x->weights); fix(l.norm2, x->weights); fix(l.shift, x->weights);
        fix(l.qkv_bias, x->weights); fix(l.conv, x->weights); fix(l.conv_b, x->weights); fix(l.dt_b, x->weights);
        fix(l.a2, x->weights); fix(l.d, x->weights);
        fix(l.ukv.w, x->weights); fix(l.q_norm, x->weights); fix(l.c_norm, x->weights);
        fix(l.turns, x->weights); fix(l.router_b, x->weights);
        if (rc == WR_CUDA_OK) rc = fix_mat(l.first, *x, x->xin, rows, x->ldw);
        if (rc == WR_CUDA_OK) rc = fix_mat(l.uq, *x, x->cq, rows, wr_ld(l.uq.k));
        if (rc == WR_CUDA_OK) rc = fix_mat(l.gate, *x, x->xin, rows, x->ldw);
        if (rc == WR_CUDA_OK) rc = fix_mat(l.router, *x, x->xin, rows, x->ldw);
        if (rc == WR_CUDA_OK && l.experts) {
            const uint32_t places = wr_route_tiles(rows, l.experts, l.top, kMoeTile) * kMoeTile;
            rc = fix_mat(l.e_up, *x, x->e_in, places, x->ldw, x->xin);
            if (rc == WR_CUDA_OK)
                rc = fix_mat(l.e_down, *x, x->e_act, places, wr_ld(l.ff), x->e_act,
                             wr_route_tiles((uint32_t)few, l.experts, l.top, 0));
        }
        if (rc == WR_CUDA_OK) rc = fix_mat(l.qkvg, *x, x->xin, rows, x->ldw);
        if (rc == WR_CUDA_OK) rc = fix_mat(l.o, *x, x->mid, rows, wr_ld(l.o.k));
        if (rc == WR_CUDA_OK) rc = fix_mat(l.in, *x, x->xin, rows, x->ldw);
        if (rc == WR_CUDA_OK) rc = fix_mat(l.x, *x, x->mid, rows, wr_ld(l.x.k));
        if (rc == WR_CUDA_OK) rc = fix_mat(l.dt, *x, x->dbc16, rows, l.dbc_ld);
        if (rc == WR_CUDA_OK) rc = fix_mat(l.out, *x, x->scan_out, rows, wr_ld(l.out.k));
        if (rc == WR_CUDA_OK) rc = fix_mat(l.up, *x, x->xin, rows, x->ldw);
        if (rc == WR_CUDA_OK) rc = fix_mat(l.down, *x, x->mid, rows, wr_ld(l.down.k));
    }
    if (rc != WR_CUDA_OK) return fail(rc);
    *out = m;
    return WR_CUDA_OK;
}

extern "C" int wr_cuda_model_kv_create(wr_cuda_ctx *ctx, wr_cuda_model *m, uint32_t max_ctx, wr_cuda_kv **out)
{
    if (!ctx || !m || m->ctx != ctx || !out) return WR_CUDA_ERR_INVAL;
    if (!m->mixed) return wr_cuda_kv_create(ctx, m->n_layers, m->n_kv, m->hd, max_ctx, out);
    return wr_cuda_kv_create_layout(ctx, (uint32_t)m->mixed->cache.size(), m->mixed->cache.data(), max_ctx, out);
}

extern "C" int wr_cuda_model_set_hidden_tap(wr_cuda_model *m, float *hidden_tap)
{
    if (!m || !m->mixed) return WR_CUDA_ERR_UNSUPPORTED;
    std::lock_guard<std::mutex> fg(m->fwd);
    m->mixed->hidden_tap = hidden_tap;
    return WR_CUDA_OK;
}

namespace {

#define TRY(expr)                               \
    do {                                        \
        const int rc__ = (expr);                \
        if (rc__ != WR_CUDA_OK) return rc__;    \
    } while (0)

// One step on its way through the stack.
struct Step {
    wr_cuda_ctx *ctx;
    wr_cuda_model *m;
    wr_mixed *x;
    wr_rows rw;
    wr_cuda_kv *const *kv;
    const uint32_t *positions;
    uint32_t max_len;
    bool wide;                           // BF16 tensor-core products (else weight-streaming ones on F32 rows)
    std::unique_lock<std::mutex> *lock;

    bool split() const { return !wide && x->compute == WR_CUDA_BF16; }
    int act() const { return wide ? WR_ACT_BF16 : WR_ACT_F32; }                              // a product's output rows
    int in_act() const { return split() ? (int)WR_ACT_SPLIT : act(); }                       // a product's input rows

    // out = act(mat . in + bias) mul + add; `in` is the buffer the matrix's row maps were made for.  Gate / up rows of
    // the matrix (BF16 models) go to pair_out.
    int product(const Mat &mat, const void *in, uint32_t in_ld, void *out, uint32_t out_ld, int out_type,
                const float *bias = nullptr, bool softplus = false, const float *add = nullptr, void *copy16 = nullptr,
                void *pair_out = nullptr, uint32_t pair_ld = 0)
    {
        const float mul = add ? x->residual_mult : 1.f;
        wr_pair_args pair = mat.pair;
        pair.out = pair_out;
        pair.ld = pair_ld;
        if (wide) {
            wr_gemm_args a{};
            a.m = rw.n_rows;
            a.out = out; a.out_ld = out_ld;
            a.out_type = out_type == WR_ACT_F32 ? WR_GEMM_OUT_F32 : out_type == WR_ACT_BF16 ? WR_GEMM_OUT_BF16 : WR_GEMM_OUT_F16;
            a.out_bf16 = copy16; a.out_bf16_ld = copy16 ? out_ld : 0;
            a.bias = bias;
            a.act = softplus ? WR_GEMM_ACT_SOFTPLUS : WR_GEMM_ACT_NONE;
            a.add = add; a.add_ld = add ? out_ld : 0;
            a.mul = mul;
            a.pair = pair;
            ++m->launches;
            return wr_gemm_launch(ctx, mat.x_map, {mat.w, mat.n, mat.k}, a);
        }
        ++m->launches;
        if (x->compute == WR_CUDA_BF16) {
            wr_skinny_args a{};
            a.rows = rw.n_rows;
            a.out = static_cast<float *>(out); a.out_ld = out_ld;
            a.out_split = copy16; a.out_split_ld = copy16 ? out_ld : 0;
            a.bias = bias;
            a.act = softplus ? WR_GEMM_ACT_SOFTPLUS : WR_GEMM_ACT_NONE;
            a.add = add; a.add_ld = out_ld;
            a.mul = mul;
            a.pair = pair;
            return wr_skinny_launch(ctx, mat.xs_map, {mat.w, mat.n, mat.k}, a);
        }
        GemvParams p{};
        p.seg[0] = {static_cast<const float *>(mat.w), static_cast<float *>(out), mat.n, out_ld};
        p.n_seg = 1;
        p.x = static_cast<const float *>(in);
        p.x_stride = in_ld;
        p.k = wr_ld(mat.k);              // the pad columns of both operands are zeros
        p.rows = rw.n_rows;
        p.add = add; p.add_stride = out_ld;
        p.bias = bias;
        p.act = softplus ? WR_GEMV_ACT_SOFTPLUS : WR_GEMV_ACT_NONE;
        p.mul = mul;
        ctx->launches++;
        return wr_gemv_launch(ctx, p, mat.n);
    }

    int norm(const float *w, const float *shift, uint64_t state_off)
    {
        wr_norm_args a{};
        a.x = x->resid; a.w = w; a.shift = shift; a.state_off = state_off;
        a.width = x->width; a.groups = x->groups; a.eps = x->eps; a.centre = x->centre;
        a.out = x->xin; a.out_type = in_act();
        ++m->launches;
        return wr_group_norm_launch(ctx, rw, a);
    }

    int attention(const Layer &l, uint32_t run)
    {
        wr_attn_geom g = l.g;
        g.layer = run;
        const int pt = wide ? WR_ACT_F16 : WR_ACT_F32;
        TRY(product(l.qkvg, x->xin, x->ldw, x->proj, l.proj_ld, pt, l.qkv_bias));
        wr_attn_prep_args p{};
        p.g = g;
        p.qkv = x->proj; p.type = pt; p.ld = l.proj_ld; p.k_off = l.k_off; p.v_off = l.v_off;
        p.scale = l.scale; p.temp_coef = l.temp_coef; p.temp_every = l.temp_every;
        p.q = x->q;
        p.q_type = g.hd128 && !rw.decode ? WR_ACT_F16 : WR_ACT_F32;
        TRY(wr_attn_prep_launch(ctx, rw, p));
        m->launches += 2;
        if (!g.hd128) {
            TRY(wr_attn_any_launch(ctx, rw, g, static_cast<const float *>(x->q), x->attn, max_len));
        } else if (rw.decode) {
            uint32_t lens[WR_CUDA_BATCH_MAX];
            for (uint32_t s = 0; s < rw.n_seq; ++s) lens[s] = positions[s] + 1;
            TRY(wr_decode_launch(ctx, rw.n_seq, kv, run, lens, static_cast<const float *>(x->q), x->attn, g.vq(), 1.0f, 0, 0,
                                 nullptr));
        } else {
            lock->unlock();
            const int rc = wr_cuda_attn_prefill(ctx, kv[0], run, positions[0], rw.n_rows, x->q, WR_CUDA_F16, x->attn, g.vq(),
                                                1.0f, 0, WR_CUDA_MEM_DEVICE);
            lock->lock();
            TRY(rc);
        }
        wr_attn_finish_args f{};
        f.g = g;
        f.o = x->attn;
        f.lambda = l.lambda; f.diff_init = l.diff_init; f.eps = l.diff_eps;
        f.gate = l.gated ? static_cast<const char *>(x->proj) + (size_t)l.g_off * (wide ? 2 : 4) : nullptr;
        f.gate_type = pt; f.gate_ld = l.proj_ld;
        f.out = x->mid; f.out_type = in_act();
        ++m->launches;
        TRY(wr_attn_finish_launch(ctx, rw, f));
        return product(l.o, x->mid, wr_ld(l.o.k), x->resid, x->ldw, WR_ACT_F32, nullptr, false, x->resid);
    }

    int mamba1(const Layer &l, uint64_t state_off)
    {
        const uint32_t ldi = wr_ld(l.inner), es = wide ? 2 : 4;
        TRY(product(l.in, x->xin, x->ldw, x->proj, 2 * ldi, act()));
        wr_conv_args c{};
        c.x = x->proj; c.type = act(); c.x_ld = 2 * ldi; c.inner = l.inner; c.taps = l.taps;
        c.w = l.conv; c.b = l.conv_b; c.state_off = state_off + l.conv_off;
        c.out = split() ? static_cast<void *>(x->conv_f32) : x->mid;
        c.out_split = split() ? x->mid : nullptr;
        TRY(wr_conv_silu_launch(ctx, rw, c));
        TRY(product(l.x, x->mid, ldi, x->dbc, l.dbc_ld, WR_ACT_F32, nullptr, false, nullptr,
                    x->compute == WR_CUDA_BF16 ? x->dbc16 : nullptr));
        TRY(product(l.dt, x->dbc, l.dbc_ld, x->dt, ldi, WR_ACT_F32, l.dt_b, true));
        wr_scan_args s{};
        s.x = c.out; s.x_ld = ldi;
        s.z = static_cast<const char *>(x->proj) + (size_t)ldi * es; s.z_ld = 2 * ldi;
        s.type = act();
        s.dt = x->dt; s.bc = x->dbc; s.bc_ld = l.dbc_ld; s.b_off = l.b_off; s.c_off = l.c_off;
        s.a2 = l.a2; s.d = l.d; s.inner = l.inner; s.state = l.state; s.state_off = state_off + l.scan_off;
        s.out = x->scan_out; s.out_type = in_act();
        TRY(wr_scan_launch(ctx, rw, s));
        m->launches += 2;
        return product(l.out, x->scan_out, ldi, x->resid, x->ldw, WR_ACT_F32, nullptr, false, x->resid);
    }

    int latent(const Layer &l, uint32_t run)
    {
        const wr_latent_geom &g = l.lat;
        wr_attn_geom ag = l.g;
        ag.layer = x->rows_of[run];
        const bool own = x->rows_of[run] == run, bf = x->compute == WR_CUDA_BF16;
        const uint32_t ld_o = wr_ld(l.o.k), es = wide || split() ? 2 : 4;
        void *ff = l.fused ? static_cast<char *>(x->mid) + (size_t)l.ff_at * es : nullptr;
        TRY(product(l.first, x->xin, x->ldw, x->lat, l.proj_ld, WR_ACT_F32, nullptr, false, nullptr, nullptr, ff, ld_o));
        if (l.fused && !bf) TRY(gate_up_f32(l, static_cast<float *>(ff), ld_o));
        wr_latent_prep_args p{};
        p.g = g; p.in = x->lat; p.ld = l.proj_ld; p.c_off = l.k_off; p.r_off = l.rot_off;
        p.q_norm = l.q_norm; p.c_norm = l.c_norm; p.eps = l.latent_eps; p.turns = l.turns;
        p.cq = x->cq; p.cq_type = in_act(); p.own = own; p.layer = run; p.kv = l.g.kv;
        wr_route_args r{};
        if (l.experts && !l.router.w) {                  // (the logits came with the first product)
            r = route_of(l, l.logit_off, l.proj_ld);
            p.route = &r;
        }
        TRY(wr_latent_prep_launch(ctx, rw, p));
        if (wide && l.flash) {
            TRY(product(l.uq, x->cq, wr_ld(g.q_rank), x->q, g.heads * g.q_head(), WR_ACT_F16));
            TRY(latent_prompt(l, ag, ld_o));
            return product(l.o, x->mid, ld_o, x->resid, x->ldw, WR_ACT_F32, nullptr, false, x->resid);
        }
        TRY(product(l.uq, x->cq, wr_ld(g.q_rank), x->q, g.heads * g.q_head(), WR_ACT_F32));
        wr_latent_query_args q{};
        q.g = g; q.q = static_cast<const float *>(x->q); q.w_ukv = l.ukv.w; q.w_type = bf ? WR_ACT_F16 : WR_ACT_F32;
        q.turns = l.turns; q.scale = l.scale; q.split = l.tensor_decode && split(); q.out = x->qa;
        TRY(wr_latent_query_launch(ctx, rw, q));
        wr_latent_value_args v{};
        v.g = g; v.o = x->olat; v.w_ukv = l.ukv.w; v.w_type = q.w_type; v.split = q.split;
        v.out = x->mid; v.out_type = in_act(); v.out_ld = ld_o;
        if (q.split) {
            uint32_t lens[WR_CUDA_BATCH_MAX];
            for (uint32_t r = 0; r < rw.n_rows; ++r) lens[r] = rw.decode ? positions[r] + 1 : positions[0] + r + 1;
            TRY(wr_latent_decode_launch(ctx, rw, g, ag.layer, x->qa, lens, x->olat, v));
            if (!v.ml) ++m->launches;
        } else {
            TRY(wr_attn_any_launch(ctx, rw, ag, x->qa, x->olat, max_len));
        }
        TRY(wr_latent_value_launch(ctx, rw, v));
        m->launches += 4;
        return product(l.o, x->mid, ld_o, x->resid, x->ldw, WR_ACT_F32, nullptr, false, x->resid);
    }

    // Keys and values of every head written out for the whole context (one product on the cached rows), then attention.
    int latent_prompt(const Layer &l, const wr_attn_geom &ag, uint32_t ld_o)
    {
        const wr_latent_geom &g = l.lat;
        const uint64_t *pages = kv[0]->d_pages + (size_t)ag.layer * kv[0]->n_pages;
        TRY(wr_latent_rotate_launch(ctx, rw, g, l.turns, x->q));
        TRY(wr_ctx_reserve_ws(ctx, (size_t)max_len * l.ukv.n * 2, 0));
        wr_gemm_args a{};
        a.m = max_len;
        a.out = ctx->ws; a.out_ld = l.ukv.n; a.out_type = WR_GEMM_OUT_F16;
        a.pages = pages;
        TRY(wr_gemm_launch(ctx, l.o.x_map, {l.ukv.w, l.ukv.n, l.ukv.k}, a));     // (the map is not read)
        wr_latent_flash_args f{};
        f.g = g; f.n = rw.n_rows; f.p0 = positions[0]; f.q = x->q; f.kv = ctx->ws; f.pages = pages; f.scale = l.scale;
        f.out = x->mid; f.out_ld = ld_o;
        m->launches += 3;
        return wr_latent_flash_launch(ctx, f);
    }

    // F32 models: silu(gate h) * (up h)
    int gate_up_f32(const Layer &l, float *out, uint32_t out_ld)
    {
        GemvParams p{};
        p.seg[0] = {static_cast<const float *>(l.gate.w), out, l.ff, out_ld};
        p.seg[1] = {static_cast<const float *>(l.up.w), nullptr, l.ff, out_ld};
        p.n_seg = 2;
        p.swiglu = 1;
        p.x = static_cast<const float *>(x->xin);
        p.x_stride = x->ldw;
        p.k = x->ldw;
        p.rows = rw.n_rows;
        ctx->launches++;
        ++m->launches;
        return wr_gemv_launch(ctx, p, l.ff);
    }

    int feed_forward(const Layer &l)
    {
        if (!l.parallel) TRY(norm(l.norm2, nullptr, 0));
        if (l.ffn == WR_CUDA_FFN_MOE) return experts(l);
        const uint32_t ld = wr_ld(l.ff);
        if (l.ffn == WR_CUDA_FFN_SWIGLU) {
            if (x->compute != WR_CUDA_BF16) TRY(gate_up_f32(l, static_cast<float *>(x->mid), ld));
            else TRY(product(l.gate, x->xin, x->ldw, nullptr, 8, WR_ACT_F32, nullptr, false, nullptr, nullptr, x->mid, ld));
        } else {
            TRY(product(l.up, x->xin, x->ldw, x->proj, ld, act()));
            wr_polynorm_args p{};
            p.z = x->proj; p.z_type = act(); p.out = x->mid; p.out_type = in_act(); p.ff = l.ff;
            p.a = l.act[0]; p.b = l.act[1]; p.c = l.act[2]; p.e = l.act[3]; p.eps = l.ffn_eps;
            ++m->launches;
            TRY(wr_polynorm_launch(ctx, rw, p));
        }
        return product(l.down, x->mid, ld, x->resid, x->ldw, WR_ACT_F32, nullptr, false, x->resid);
    }

    // Router logits in columns off .. of lat.
    wr_route_args route_of(const Layer &l, uint32_t off, uint32_t ld) const
    {
        wr_route_args r{};
        r.logits = x->lat + off; r.ld = ld; r.bias = l.router_b; r.experts = l.experts; r.top = l.top;
        r.tile = split() ? 0 : x->compute == WR_CUDA_BF16 ? kMoeTile : kMoeTileF32;
        r.weight = x->e_weight; r.expert = x->e_expert; r.place = x->e_place; r.row_of = x->e_row_of;
        r.list = x->e_list; r.count = x->e_count;
        return r;
    }

    int experts(const Layer &l)
    {
        const bool bf = x->compute == WR_CUDA_BF16;
        wr_route_args r = route_of(l, l.logit_off, l.proj_ld);
        if (l.router.w) {
            r = route_of(l, 0, wr_ld(l.experts));
            TRY(product(l.router, x->xin, x->ldw, x->lat, r.ld, WR_ACT_F32));
        } else {
            r.chosen = true;                             // (by wr_latent_prep_launch)
        }
        TRY(wr_route_launch(ctx, rw, r));
        const uint32_t groups = wr_route_tiles(rw.n_rows, l.experts, l.top, r.tile), lf = wr_ld(l.ff);
        wr_group_args gr;
        gr.list = x->e_list; gr.count = x->e_count; gr.max = groups; gr.usual = l.top;
        wr_combine_args c{};
        if (split()) {
            wr_skinny_args a{};
            a.rows = rw.n_rows;
            a.pair = l.e_up.pair; a.pair.out = x->e_act; a.pair.ld = lf;
            a.group = gr; a.group.stride = l.up_stride;
            TRY(wr_skinny_launch(ctx, l.e_up.xs_map, {l.e_up.w, l.e_up.n, l.e_up.k}, a));
            wr_skinny_args b{};
            b.rows = rw.n_rows;
            b.out = static_cast<float *>(x->e_out); b.out_ld = x->ldw;
            b.group = gr; b.group.stride = l.down_stride; b.group.x_rows = 2 * WR_CUDA_BATCH_MAX;
            TRY(wr_skinny_launch(ctx, l.e_down.xs_map, {l.e_down.w, l.e_down.n, l.e_down.k}, b));
            c.type = WR_ACT_F32;
            c.few = true;
        } else if (bf) {
            TRY(wr_moe_gather_launch(ctx, x->xin, x->e_in, x->ldw, x->e_row_of, x->e_count, groups, kMoeTile));
            wr_gemm_args a{};
            a.m = groups * kMoeTile;
            a.pair = l.e_up.pair; a.pair.out = x->e_act; a.pair.ld = lf;
            a.group = gr; a.group.stride = l.up_stride;
            TRY(wr_gemm_launch(ctx, l.e_up.x_map, {l.e_up.w, l.e_up.n, l.e_up.k}, a));
            wr_gemm_args b{};
            b.m = groups * kMoeTile;
            b.out = x->e_out; b.out_ld = x->ldw; b.out_type = WR_GEMM_OUT_BF16;
            b.group = gr; b.group.stride = l.down_stride;
            TRY(wr_gemm_launch(ctx, l.e_down.x_map, {l.e_down.w, l.e_down.n, l.e_down.k}, b));
            c.type = WR_ACT_BF16;
            ++m->launches;
        } else {
            wr_moe_f32_args a{};
            a.x = static_cast<const float *>(x->xin); a.x_ld = x->ldw; a.n = l.ff; a.k = x->width;
            a.gate = static_cast<const float *>(l.e_up.w); a.up = a.gate + l.up_at; a.stride = l.up_stride / 4;
            a.row_of = x->e_row_of; a.list = x->e_list; a.count = x->e_count; a.max_tiles = groups;
            a.alpha = l.alpha; a.limit = l.limit;
            a.out = static_cast<float *>(x->e_act); a.out_ld = lf;
            TRY(wr_moe_f32_launch(ctx, a));
            wr_moe_f32_args b = a;
            b.x = a.out; b.x_ld = lf; b.n = x->width; b.k = l.ff; b.row_of = nullptr;
            b.gate = static_cast<const float *>(l.e_down.w); b.up = nullptr; b.stride = l.down_stride / 4;
            b.out = static_cast<float *>(x->e_out); b.out_ld = x->ldw;
            TRY(wr_moe_f32_launch(ctx, b));
            c.type = WR_ACT_F32;
        }
        c.y = x->e_out; c.ld = x->ldw; c.width = x->width; c.top = l.top; c.weight = x->e_weight; c.place = x->e_place;
        c.mul = x->residual_mult; c.resid = x->resid;
        m->launches += 4;
        return wr_moe_combine_launch(ctx, rw, c);
    }
};

}  // namespace

int wr_mixed_forward(wr_cuda_ctx *ctx, wr_cuda_model *m, int mode, uint32_t n_rows, wr_cuda_kv *const *kv,
                     const uint32_t *positions, const uint32_t *tokens, uint32_t out_from, float *hidden_out,
                     float *normed_out, float *const *logits_out, uint32_t *argmax_out)
{
    wr_mixed *x = m->mixed;
    const bool decode = mode == WR_CUDA_FWD_DECODE;
    if (n_rows == 0 || n_rows > m->max_rows || out_from > n_rows) return WR_CUDA_ERR_LIMIT;
    if (decode && n_rows > WR_CUDA_BATCH_MAX) return WR_CUDA_ERR_LIMIT;
    const uint32_t n_out = n_rows - out_from, n_seq = decode ? n_rows : 1, per_seq = decode ? 1 : n_rows;
    if (argmax_out && n_out > WR_CUDA_BATCH_MAX) return WR_CUDA_ERR_LIMIT;
    if ((normed_out || logits_out || argmax_out) && n_out == 0) return WR_CUDA_ERR_INVAL;
    for (uint32_t r = 0; r < n_rows; ++r)
        if (tokens[r] >= m->vocab) return WR_CUDA_ERR_INVAL;      // refused before anything runs

    std::lock_guard<std::mutex> fg(m->fwd);
    const auto t_begin = std::chrono::steady_clock::now();
    std::unique_lock<std::mutex> lock(ctx->lock);
    WR_CUDA_TRY(cudaSetDevice(ctx->device));
    int slot_out[WR_CUDA_BATCH_MAX];
    uint32_t max_len = 0;
    for (uint32_t s = 0; s < n_seq; ++s) {
        if (!kv[s] || kv[s]->ctx != ctx || kv[s]->n_layers != x->cache.size() || kv[s]->state_bytes != x->state_bytes)
            return WR_CUDA_ERR_INVAL;
        for (uint32_t t = 0; t < s; ++t)
            if (kv[t] == kv[s]) return WR_CUDA_ERR_INVAL;
        for (uint32_t i = 0; i < kv[s]->n_layers; ++i) {
            const wr_kv_geom &a = kv[s]->layers[i].geom;
            const wr_cuda_cache_layer &b = x->cache[i];
            if (a.n_kv != b.n_kv_heads || (a.n_kv && (a.k_dim != b.k_dim || a.v_dim != b.v_dim || a.elem != b.elem)))
                return WR_CUDA_ERR_INVAL;
        }
        if ((uint64_t)positions[s] + per_seq > kv[s]->max_ctx) return WR_CUDA_ERR_CTX_FULL;
        if ((uint64_t)positions[s] + per_seq > ctx->attn_max_seq) return WR_CUDA_ERR_LIMIT;
        max_len = std::max(max_len, positions[s] + per_seq);
    }
    for (uint32_t s = 0; s < n_seq; ++s) {
        const bool fresh = positions[s] == 0;
        const int in = fresh ? 1 : kv[s]->state_slot(positions[s]);
        if (x->state_bytes && in < 0) return WR_CUDA_ERR_STATE;
        wr_seq_dev &q = x->h_seqs[s];
        q.pages = kv[s]->d_pages;
        slot_out[s] = x->state_bytes ? 1 - in : 0;
        q.st_in = x->state_bytes ? static_cast<const char *>(kv[s]->state[in]) : nullptr;
        q.st_out = x->state_bytes ? static_cast<char *>(kv[s]->state[1 - in]) : nullptr;
        q.pos = positions[s];
        q.n = per_seq;
        q.fresh = fresh ? 1u : 0u;
        q.n_pages = kv[s]->n_pages;
    }
    // from here on the slots being written hold nothing until the step has succeeded
    for (uint32_t s = 0; s < n_seq; ++s) {
        kv[s]->state_len[slot_out[s]] = -1;
        if (positions[s] == 0) kv[s]->state_len[1 - slot_out[s]] = -1;
    }
    cudaStream_t st = ctx->stream;
    memcpy(x->h_tokens, tokens, n_rows * sizeof(uint32_t));
    WR_CUDA_TRY(cudaMemcpyAsync(x->tokens, x->h_tokens, n_rows * sizeof(uint32_t), cudaMemcpyHostToDevice, st));
    WR_CUDA_TRY(cudaMemcpyAsync(x->seqs, x->h_seqs, n_seq * sizeof(wr_seq_dev), cudaMemcpyHostToDevice, st));

    const bool bf = x->compute == WR_CUDA_BF16;
    Step step{};
    step.ctx = ctx; step.m = m; step.x = x; step.kv = kv; step.positions = positions; step.max_len = max_len;
    step.rw = {x->seqs, n_rows, n_seq, decode ? 1u : 0u};
    step.wide = bf && n_rows > WR_CUDA_BATCH_MAX;
    step.lock = &lock;
    TRY(wr_embed_launch(ctx, step.rw, x->tokens, x->embed, bf ? WR_ACT_BF16 : WR_ACT_F32, x->turns, x->resid, x->width, x->embed_scale));
    ++m->launches;
    const size_t row_bytes = (size_t)x->width * 4, ld_bytes = (size_t)x->ldw * 4;
    for (uint32_t i = 0; i < x->runs.size(); ++i) {
        const Layer &l = x->layers[x->runs[i]];
        TRY(step.norm(l.norm1, l.shift, x->state_off[i]));
        if (l.mixer == WR_CUDA_MIXER_ATTENTION) TRY(step.attention(l, i));
        else if (l.mixer == WR_CUDA_MIXER_LATENT) TRY(step.latent(l, i));
        else TRY(step.mamba1(l, x->state_off[i]));
        if (l.ffn != WR_CUDA_FFN_NONE && !l.fused) TRY(step.feed_forward(l));
        if (x->hidden_tap)
            WR_CUDA_TRY(cudaMemcpy2DAsync(x->hidden_tap + (size_t)i * n_rows * x->width, row_bytes, x->resid, ld_bytes,
                                          row_bytes, n_rows, cudaMemcpyDeviceToHost, st));
    }
    if (hidden_out && n_out)
        WR_CUDA_TRY(cudaMemcpy2DAsync(hidden_out, row_bytes, x->resid + (size_t)out_from * x->ldw, ld_bytes, row_bytes, n_out,
                                      cudaMemcpyDeviceToHost, st));
    // The rows somebody asked for, in passes of kHeadRows: final norm, head, copies out.
    uint32_t n_want = 0;
    for (uint32_t i = 0; i < n_out; ++i)
        if (normed_out || argmax_out || (logits_out && logits_out[i])) x->h_gather[n_want++] = out_from + i;
    if (n_want) {
        const uint32_t ldv = wr_ld(m->vocab);
        WR_CUDA_TRY(cudaMemcpyAsync(x->gather, x->h_gather, n_want * sizeof(uint32_t), cudaMemcpyHostToDevice, st));
        for (uint32_t done = 0; done < n_want; done += kHeadRows) {
            Step head = step;
            head.rw.n_rows = std::min(kHeadRows, n_want - done);
            head.wide = bf && head.rw.n_rows > WR_CUDA_BATCH_MAX;
            wr_norm_args a{};
            a.x = x->resid; a.gather = x->gather + done; a.w = x->final_norm;
            a.width = x->width; a.groups = x->groups; a.eps = x->eps; a.centre = x->centre;
            a.out = x->head_in; a.out_type = head.in_act();
            if (logits_out || argmax_out) {
                TRY(wr_group_norm_launch(ctx, head.rw, a));
                TRY(head.product(x->head, x->head_in, x->ldw, x->logits, ldv, WR_ACT_F32));
                ++m->launches;
            }
            if (normed_out) {
                a.out = x->normed;
                a.out_type = WR_ACT_F32;
                TRY(wr_group_norm_launch(ctx, head.rw, a));
                ++m->launches;
                WR_CUDA_TRY(cudaMemcpy2DAsync(normed_out + (size_t)done * x->width, row_bytes, x->normed, ld_bytes, row_bytes,
                                              head.rw.n_rows, cudaMemcpyDeviceToHost, st));
            }
            if (argmax_out) {
                TRY(wr_argmax_launch(st, x->logits, ldv, m->vocab, head.rw.n_rows, x->part_v, x->part_i, x->best));
                ctx->launches += 2;
                m->launches += 2;
                WR_CUDA_TRY(cudaMemcpyAsync(x->h_best, x->best, head.rw.n_rows * sizeof(uint32_t), cudaMemcpyDeviceToHost, st));
            }
            for (uint32_t i = 0; logits_out && i < head.rw.n_rows; ++i) {
                float *dst = logits_out[x->h_gather[done + i] - out_from];
                if (dst)
                    WR_CUDA_TRY(cudaMemcpyAsync(dst, x->logits + (size_t)i * ldv, (size_t)m->vocab * 4,
                                                cudaMemcpyDeviceToHost, st));
            }
        }
    }
    m->last_enqueue_ns = (uint64_t)std::chrono::duration_cast<std::chrono::nanoseconds>(
                             std::chrono::steady_clock::now() - t_begin).count();
    TRY(wr_ctx_sync_checked(ctx));
    for (uint32_t s = 0; s < n_seq; ++s) kv[s]->state_len[slot_out[s]] = (int64_t)positions[s] + per_seq;
    if (argmax_out)
        for (uint32_t i = 0; i < n_out; ++i) argmax_out[i] = x->h_best[i];
    return WR_CUDA_OK;
}
