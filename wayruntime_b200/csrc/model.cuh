// model.cuh — wr_cuda_model: the F32 layer stack of model_glue.cu or the mixed stack of model_mixed.cu.
#pragma once

#include "wr_internal.cuh"

struct wr_cuda_layer_dev {
    const float *attn_norm, *wq, *wk, *wv, *q_norm, *k_norm, *wo, *ffn_norm, *w_gate, *w_up, *w_down;
    uint32_t ffn;
};

struct wr_mixed;                         // model_mixed.cu

struct wr_cuda_model {
    wr_cuda_ctx *ctx = nullptr;
    wr_mixed *mixed = nullptr;           // set: the mixed stack, and nothing but ctx / vocab / counters below is used
    uint32_t n_layers = 0, hidden = 0, n_q = 0, n_kv = 0, hd = 0, vocab = 0, n_rot = 0, max_rows = 0;
    float eps = 0.f, theta = 0.f, scale = 0.f;
    char *slab = nullptr;                // every weight, one allocation
    size_t slab_bytes = 0;
    const float *embed = nullptr, *lm_head = nullptr, *final_norm = nullptr;
    std::vector<wr_cuda_layer_dev> layers;
    // row scratch (device)
    float *resid = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *attn = nullptr, *gate = nullptr;
    float *normed = nullptr, *logits = nullptr;
    uint32_t *tokens = nullptr, *best = nullptr, *part_i = nullptr;
    float *part_v = nullptr;             // arg-max partials [16][kArgmaxParts]
    uint32_t *h_tokens = nullptr;        // pinned: token ids in, arg-max ids out
    uint32_t ffn_max = 0;
    uint64_t launches = 0;
    uint64_t last_enqueue_ns = 0;        // host time the last forward pass spent before it began to wait
    std::mutex fwd;                      // one forward pass at a time (the scratch rows are shared)
};

// First maximum of `rows` logit rows (stride ld) -> best[row]; part_v / part_i: WR_ARGMAX_PARTS entries per row.
constexpr int WR_ARGMAX_PARTS = 64;
int wr_argmax_launch(cudaStream_t st, const float *logits, uint32_t ld, uint32_t vocab, uint32_t rows, float *part_v,
                     uint32_t *part_i, uint32_t *best);

int  wr_mixed_forward(wr_cuda_ctx *ctx, wr_cuda_model *m, int mode, uint32_t n_rows, wr_cuda_kv *const *kv,
                      const uint32_t *positions, const uint32_t *tokens, uint32_t out_from, float *hidden_out,
                      float *normed_out, float *const *logits_out, uint32_t *argmax_out);
void wr_mixed_destroy(wr_mixed *x);      // caller holds ctx->lock, device current, stream idle
