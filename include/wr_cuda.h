/*
 * wr_cuda.h — C-ABI of the B200 (sm_100a) attention hot path for wayruntime.
 *
 * This is the seam the reference's C11 host code (src/core/session.c,
 * src/core/batch.c) calls in place of its CPU ops:
 *
 *   wr_cuda_kv_append     <- wri_op_rope on Q and K + kv_append_row on K and V
 *                            (src/core/session.c:471-487, kernels.c:1356,
 *                             session.c:139)
 *   wr_cuda_attn_decode   <- wri_op_gqa_attention with seq_q = 1, once per
 *                            session (src/core/session.c:490-496,
 *                             kernels.c:1414; batched: batch.c:152-164)
 *   wr_cuda_attn_prefill  <- the wri_session_prefill loop of single-token
 *                            attention calls (src/core/session.c:599-630)
 *
 * Plain pointers and sizes only.  Every function returns a wr_status value
 * (include/wayruntime/wayruntime.h:82-107): 0 or a negative code; nothing
 * aborts, prints or falls back to the CPU.  There is no CPU path: without an
 * sm_100 device every entry point fails with WR_CUDA_ERR_UNSUPPORTED.
 *
 * Threading: a context serialises its own calls with a mutex, so distinct
 * sessions may be driven from distinct threads (wayruntime.h:29-40).
 */
#ifndef WR_CUDA_H
#define WR_CUDA_H

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* wr_status values used here (wayruntime.h:82-107). */
#define WR_CUDA_OK               0
#define WR_CUDA_ERR_UNSUPPORTED (-3)
#define WR_CUDA_ERR_INVAL       (-4)
#define WR_CUDA_ERR_NOMEM       (-5)
#define WR_CUDA_ERR_CTX_FULL    (-6)
#define WR_CUDA_ERR_STATE       (-7)
#define WR_CUDA_ERR_LIMIT       (-8)
#define WR_CUDA_ERR_INTERNAL    (-10)

/* Where the caller's Q / K / V / output buffers live. */
#define WR_CUDA_MEM_HOST   0   /* host memory; the call copies and synchronises */
#define WR_CUDA_MEM_DEVICE 1   /* device memory; the call only enqueues */

/* Element types (values of wr_dtype, src/core/internal.h:53-55). */
#define WR_CUDA_F32 0
#define WR_CUDA_F16 1
#define WR_CUDA_BF16 2     /* weights and the matrix products of wr_cuda_model_create_mixed only */

/* wr_cuda_kv_append flags. */
#define WR_CUDA_APPEND_ROPE 1u  /* rotate K (and Q when given) before storing */

#define WR_CUDA_BATCH_MAX        16    /* WR_BATCH_MAX, wayruntime.h:423 */
#define WR_CUDA_ATTN_MAX_SEQ     4096  /* default cap, WR_ATTN_MAX_SEQ (internal.h:186) */
#define WR_CUDA_ATTN_MAX_SEQ_TOP 1048576
#define WR_CUDA_HEAD_DIM_MAX     1024  /* WR_FLASH_D_MAX (internal.h:197) */
#define WR_CUDA_PAGE_TOKENS      64    /* tokens per KV page = WR_FLASH_BLOCK */
#define WR_CUDA_TRIPLE_PAD       4     /* floats before o[] in a split-KV triple */

typedef struct wr_cuda_ctx wr_cuda_ctx;  /* one device, one stream, one page pool */
typedef struct wr_cuda_kv  wr_cuda_kv;   /* one session's paged F16 K/V cache   */

/* ---- device / context -------------------------------------------------- */

/* WR_CUDA_OK when `device` exists and is compute capability 10.x.  This is
 * the check wr_engine_create makes beside its endian probe
 * (src/core/engine.c:130): no B200 bound -> WR_ERR_UNSUPPORTED. */
int wr_cuda_device_check(int device);

int  wr_cuda_ctx_create(int device, wr_cuda_ctx **out);
void wr_cuda_ctx_destroy(wr_cuda_ctx *ctx);

/* Wait for everything enqueued on the context's stream.  Also reports (and
 * clears) a device-side error flag: a bounded wait that gave up inside a
 * kernel surfaces here — and at the end of every call that takes
 * WR_CUDA_MEM_HOST buffers — as WR_CUDA_ERR_INTERNAL. */
int  wr_cuda_ctx_sync(wr_cuda_ctx *ctx);

/* The context's cudaStream_t, for callers that time or order against it. */
void *wr_cuda_ctx_stream(wr_cuda_ctx *ctx);

/* Sequence cap for sessions and attention calls on this context; the
 * reference's WR_ATTN_MAX_SEQ is a compile-time constant (internal.h:186),
 * here it is a setting so long-context shards need no rebuild. */
int  wr_cuda_ctx_set_attn_max_seq(wr_cuda_ctx *ctx, uint32_t max_seq);

/* Every device-side wait in this library (an mbarrier phase, an arrival
 * counter, a peer's flag) gives up after this many cycles of SM clock: the
 * kernel records an error word, unwinds and returns, and the next call that
 * synchronises (wr_cuda_ctx_sync, or any call with WR_CUDA_MEM_HOST buffers)
 * returns WR_CUDA_ERR_INTERNAL once and clears the word; the context stays
 * usable.  The reference has no counterpart (its ops cannot stall); the
 * contract kept is its "a failed step consumes nothing" (session.c:160-168,
 * :589-592).  Default WR_CUDA_WAIT_LIMIT_DEFAULT, about two seconds. */
#define WR_CUDA_WAIT_LIMIT_DEFAULT 4000000000LL
int  wr_cuda_ctx_set_wait_limit(wr_cuda_ctx *ctx, int64_t cycles);
/* The error word of the last give-up reported (0: none yet): a small number
 * naming the wait that ran out, for a log line next to WR_CUDA_ERR_INTERNAL. */
int  wr_cuda_ctx_last_device_error(wr_cuda_ctx *ctx);

/* Page-locked host memory for a caller's row buffers (Q / K / V / attention
 * rows): with such buffers the WR_CUDA_MEM_HOST calls need no staging copy —
 * the decode kernels read and write them in place.  The reference's session
 * scratch comes from one arena sized at create (session.c:699-708); a host
 * layer allocates these once per session in the same place and frees them at
 * destroy.  64-byte aligned.  WR_CUDA_ERR_NOMEM when the host cannot pin. */
int  wr_cuda_host_alloc(wr_cuda_ctx *ctx, uint64_t bytes, void **out);
void wr_cuda_host_free(wr_cuda_ctx *ctx, void *p);

/* Number of kernels this library has launched on the context so far. */
uint64_t wr_cuda_ctx_launch_count(wr_cuda_ctx *ctx);

/* ---- KV cache (session_build / wr_session_create, session.c:640-814) ---- */

/* All pages of the session are taken from the context's pool here, once:
 * no allocation happens during decode.  max_ctx above the context's cap is
 * WR_CUDA_ERR_LIMIT (session.c:755). */
int  wr_cuda_kv_create(wr_cuda_ctx *ctx, uint32_t n_layers, uint32_t n_kv_heads,
                       uint32_t head_dim, uint32_t max_ctx, wr_cuda_kv **out);
/* The same for a model whose layers keep different things (no reference
 * counterpart: every layer of the reference keeps F16 rows of one head_dim,
 * session.c:647-674).  Per layer: K/V pages of n_kv_heads heads with rows of
 * k_dim and v_dim elements of `elem` (WR_CUDA_F32 or WR_CUDA_F16; n_kv_heads 0:
 * none), and state_bytes of recurrent state (0: none).  v_dim 0: one row per token
 * and head that serves as key and value (a multiple of 64 elements when F16).
 * Layers with F16 rows and k_dim = v_dim have the page layout of wr_cuda_kv_create and are accepted by
 * every call below; other layers by wr_cuda_model_forward only. */
#define WR_CUDA_MAX_LAYER_RUNS 1024
typedef struct wr_cuda_cache_layer {
    uint32_t n_kv_heads, k_dim, v_dim, elem;
    uint64_t state_bytes;
} wr_cuda_cache_layer;
int  wr_cuda_kv_create_layout(wr_cuda_ctx *ctx, uint32_t n_layers, const wr_cuda_cache_layer *layers,
                              uint32_t max_ctx, wr_cuda_kv **out);
void wr_cuda_kv_destroy(wr_cuda_kv *kv);
uint32_t wr_cuda_kv_max_ctx(const wr_cuda_kv *kv);

/* Copy rows [row0, row0+n) of one layer's K (which=0) or V (which=1) between
 * the paged cache and a [n, n_kv_heads, head_dim] F16 buffer in the
 * reference's row layout (session.c:647-674).  Used to load a prepared cache
 * and to compare cache bytes with the reference's. */
int wr_cuda_kv_write_rows(wr_cuda_ctx *ctx, wr_cuda_kv *kv, uint32_t layer,
                          int which, uint32_t row0, uint32_t n,
                          const uint16_t *src, int mem);
int wr_cuda_kv_read_rows(wr_cuda_ctx *ctx, wr_cuda_kv *kv, uint32_t layer,
                         int which, uint32_t row0, uint32_t n, uint16_t *dst,
                         int mem);

/* ---- the hot path -------------------------------------------------------- */

/* Fused RoPE + KV append for one layer.  Session s contributes n_tokens
 * consecutive rows at cache rows positions[s] .. positions[s]+n_tokens-1
 * (its absolute positions).  k_rows, v_rows: F32 [n_sess*n_tokens,
 * n_kv_heads, head_dim].  With WR_CUDA_APPEND_ROPE, K is rotated with the
 * reference's RoPE (kernels.c:1356-1412: its polynomial sin/cos, pairing j
 * with j+head_dim/2, n_rot_pairs as there) and q_rows — F32
 * [n_sess*n_tokens, n_q_heads, head_dim], may be NULL — is rotated in place.
 * K and V are stored with the reference's truncating F32->F16
 * (quant.c:121-136), so cache bytes equal the reference's.
 * The call does not move any committed length: the host passes seq_lens to
 * the attention calls and simply does not advance them when a step fails
 * (wri_session_kv_rollback, session.c:160).  A row past max_ctx is
 * WR_CUDA_ERR_CTX_FULL before anything is launched (session.c:144). */
int wr_cuda_kv_append(wr_cuda_ctx *ctx, uint32_t n_sess, wr_cuda_kv *const *kv,
                      uint32_t layer, const uint32_t *positions,
                      uint32_t n_tokens, const float *k_rows,
                      const float *v_rows, float *q_rows, uint32_t n_q_heads,
                      float theta_base, uint32_t n_rot_pairs, uint32_t flags,
                      int mem);

/* Decode attention, all sessions in one grid.  q, out: F32 [n_sess,
 * n_q_heads, head_dim] (q already rotated, e.g. by wr_cuda_kv_append).
 * seq_lens[s] = rows of session s to attend (the row just appended
 * included).  scale_override <= 0 selects 1/sqrt(head_dim); window > 0
 * keeps the last `window` keys (kernels.c:1456-1464).  Validation follows
 * kernels.c:1418-1454.  A session's result does not depend on which other
 * sessions share the call. */
int wr_cuda_attn_decode(wr_cuda_ctx *ctx, uint32_t n_sess,
                        wr_cuda_kv *const *kv, uint32_t layer,
                        const uint32_t *seq_lens, const float *q, float *out,
                        uint32_t n_q_heads, float scale_override,
                        uint32_t window, int mem);

/* The batched decode layer-step in one call: wr_cuda_kv_append with
 * n_tokens = 1 followed by wr_cuda_attn_decode over seq_lens[s] =
 * positions[s] + 1 — the per-layer body of wri_batch_decode_step
 * (src/core/batch.c:152-164 -> session.c:471-496) for all sessions at once.
 * q: F32 [n_sess, n_q_heads, head_dim], un-rotated on entry (rotated in
 * place when it is device memory); out: F32 of the same shape.  With host
 * buffers q, k_rows and v_rows cross the bus once and only out comes back;
 * page-locked host buffers are read and written by the kernels themselves (no
 * copy operations), pageable ones are staged.  Host q rows are left as given. */
int wr_cuda_decode_step(wr_cuda_ctx *ctx, uint32_t n_sess, wr_cuda_kv *const *kv,
                        uint32_t layer, const uint32_t *positions, float *q,
                        const float *k_rows, const float *v_rows, float *out,
                        uint32_t n_q_heads, float theta_base, uint32_t n_rot_pairs,
                        uint32_t flags, float scale_override, uint32_t window,
                        int mem);

/* Decode attention that never allocates.  (No counterpart in the reference:
 * its attention op mallocs a scratch row on every call, kernels.c:1471.)
 * Same arguments, checks and result as wr_cuda_attn_decode with device
 * buffers, but the split-KV scratch lives in a fixed array inside the library
 * image instead of buffers the context grows on demand.  It is meant for
 * callers that may not allocate at step time — a serving loop whose device
 * memory is fully committed to the KV pool, a thread that must not enter the
 * CUDA allocator.  head_dim 128 only; q and out are device memory; a call
 * needing more than WR_CUDA_STATIC_MAX_ITEMS work items (sessions x kv heads
 * x key chunks) or WR_CUDA_STATIC_MAX_GROUPS groups is WR_CUDA_ERR_LIMIT.
 * The first call on a device resolves the array's address: make it before
 * opening a stream capture.  All calls share the one array per device, so
 * calls that overlap on the GPU race; issue them one after another. */
#define WR_CUDA_STATIC_MAX_ITEMS  4096
#define WR_CUDA_STATIC_MAX_GROUPS 1024
int wr_cuda_attn_decode_static(wr_cuda_ctx *ctx, uint32_t n_sess,
                               wr_cuda_kv *const *kv, uint32_t layer,
                               const uint32_t *seq_lens, const float *q,
                               float *out, uint32_t n_q_heads,
                               float scale_override, uint32_t window);

/* Causal prefill attention for n new tokens of one session whose rows
 * [0, p0+n) are already in the cache: query i attends rows [0, p0+i]
 * (row i of the reference's prefill loop, session.c:599-630).
 * q: [n, n_q_heads, head_dim] of q_dtype; out: F32 of the same shape. */
int wr_cuda_attn_prefill(wr_cuda_ctx *ctx, wr_cuda_kv *kv, uint32_t layer,
                         uint32_t p0, uint32_t n, const void *q, int q_dtype,
                         float *out, uint32_t n_q_heads, float scale_override,
                         uint32_t window, int mem);

/* ---- split-KV across devices --------------------------------------------- */

/* Like wr_cuda_attn_decode over this device's shard of each session's keys,
 * but emits one triple per (session, q head) instead of the normalised row:
 * triples is F32 [n_sess, n_q_heads, WR_CUDA_TRIPLE_PAD + head_dim] holding
 * (m, l, 0, 0, o[head_dim]) with m the running max (natural-log domain,
 * -1e30 for an empty shard), l the denominator and o the unnormalised
 * accumulator — the state of kernels.c:1480-1516 after the shard's keys.
 * seq_lens[s] may be 0 (empty shard). */
int wr_cuda_attn_decode_partial(wr_cuda_ctx *ctx, uint32_t n_sess,
                                wr_cuda_kv *const *kv, uint32_t layer,
                                const uint32_t *seq_lens, const float *q,
                                float *triples, uint32_t n_q_heads,
                                float scale_override, int mem);

/* Merge n_shards triples per row with the online-softmax rule
 * (kernels.c:1503-1506 applied across shards): triples is F32 [n_shards,
 * n_rows, WR_CUDA_TRIPLE_PAD + head_dim], out F32 [n_rows, head_dim]. */
int wr_cuda_attn_combine(wr_cuda_ctx *ctx, uint32_t n_shards, uint32_t n_rows,
                         uint32_t head_dim, const float *triples, float *out,
                         int mem);

/* ---- Peer exchange for key-sharded decode (no reference counterpart: the
 * reference is single-device; this is the multi-GPU form of the merge above).
 *
 * One process per GPU.  Every rank creates an exchange object (a device
 * buffer for world x max_rows triples, twice, plus flags), publishes its
 * handle (WR_CUDA_XCHG_HANDLE_BYTES opaque bytes, valid in other processes of
 * this machine), receives everybody's handles in rank order by whatever
 * transport the host has, and connects: the peers' buffers are then mapped
 * over NVLink.  WR_CUDA_ERR_UNSUPPORTED when two of the devices cannot reach
 * each other's memory. */
typedef struct wr_cuda_xchg wr_cuda_xchg;
#define WR_CUDA_XCHG_MAX_WORLD    8
#define WR_CUDA_XCHG_HANDLE_BYTES 64

int  wr_cuda_xchg_create(wr_cuda_ctx *ctx, uint32_t world, uint32_t rank,
                         uint32_t max_rows, uint32_t head_dim, wr_cuda_xchg **out);
int  wr_cuda_xchg_handle(wr_cuda_xchg *x, void *handle_out);
int  wr_cuda_xchg_connect(wr_cuda_xchg *x, const void *handles /* world x 64 bytes */);
/* The same connection for exchange objects that live in ONE process (one
 * thread per GPU, or several contexts of a test): all[r] is rank r's object;
 * devices other than the caller's need peer access enabled by the host. */
int  wr_cuda_xchg_connect_local(wr_cuda_xchg *x, wr_cuda_xchg *const *all);
/* Destroy is collective: a peer's kernel may still be storing into this
 * rank's buffer, so every rank first synchronises its context
 * (wr_cuda_ctx_sync, also after a step that timed out) and the ranks agree
 * (a barrier of the host's transport) before any of them destroys. */
void wr_cuda_xchg_destroy(wr_cuda_xchg *x);

/* All-gather + merge in one kernel: stores this rank's triples (device, F32
 * [n_rows, WR_CUDA_TRIPLE_PAD + head_dim], as written by
 * wr_cuda_attn_decode_partial) into every rank's buffer, waits (bounded; an
 * expired wait surfaces at wr_cuda_ctx_sync as WR_CUDA_ERR_INTERNAL) for every
 * rank's triples of the same step, and merges them in rank order into out
 * (device, F32 [n_rows, head_dim]).  Every rank must make the same sequence of
 * calls with the same n_rows.  Enqueues on the context's stream and returns. */
int wr_cuda_attn_exchange_combine(wr_cuda_ctx *ctx, wr_cuda_xchg *x, uint32_t n_rows,
                                  const float *triples, float *out);

/* Key-sharded decode with the exchange fused into the decode kernel (no
 * reference counterpart, as above): wr_cuda_attn_decode_partial and
 * wr_cuda_attn_exchange_combine in one call.  The decode kernel's own warps
 * store every finished (session, q head) triple into all ranks' buffers,
 * flag each row there, wait (bounded) for the same rows from every rank and
 * merge them in rank order into out (device, F32 [n_sess, n_q_heads,
 * head_dim]) — one kernel.  Where a session of this rank has fewer than two
 * key chunks (a short or empty shard) the rows are published per step instead
 * and a small second kernel does the waiting and merging.  q is device
 * memory; head_dim 128.  Identical bits to the two-call sequence.  Every rank
 * makes the same sequence of calls. */
int wr_cuda_attn_decode_exchange(wr_cuda_ctx *ctx, wr_cuda_xchg *x, uint32_t n_sess,
                                 wr_cuda_kv *const *kv, uint32_t layer,
                                 const uint32_t *seq_lens, const float *q, float *out,
                                 uint32_t n_q_heads, float scale_override);

/* ---- the layer stack around attention, device-resident ------------------- */

/* A device copy of one model's F32 weights plus the row scratch of a forward
 * pass.  Replaces, for the callers of attention, the host loop of the
 * reference's decode body (src/core/session.c:405-568: RMSNorm, Q/K/V
 * projections, per-head QK-norm, attention, output projection, residual,
 * RMSNorm, SwiGLU FFN, residual; then final RMSNorm and LM head,
 * session.c:540-560) so that a row enters the device as a token id and leaves
 * as logits instead of crossing the bus twice per layer.  Llama / Qwen3-class
 * layers only (no sandwich norms, no per-layer embeddings).
 *
 * Weights are host pointers to F32 data in the GGML layout the reference keeps
 * them in: a [in -> out] projection is out rows of in floats
 * (src/core/kernels.c:978-1000).  embed and lm_head are [vocab][hidden]; they
 * may be the same pointer (tied), and are then uploaded once. */
#define WR_CUDA_MAX_LAYERS  64   /* WR_MAX_LAYERS, src/core/internal.h:184 */
#define WR_CUDA_FWD_DECODE  0    /* row r = next token of session kv[r] at positions[r] */
#define WR_CUDA_FWD_PREFILL 1    /* rows = consecutive tokens of kv[0] from positions[0] */

typedef struct wr_cuda_model wr_cuda_model;

typedef struct wr_cuda_layer_desc {
    const float *attn_norm;           /* [hidden] */
    const float *wq, *wk, *wv;        /* [n_q*hd][hidden], [n_kv*hd][hidden] x2 */
    const float *q_norm, *k_norm;     /* [head_dim] each, or both NULL */
    const float *wo;                  /* [hidden][n_q*hd] */
    const float *ffn_norm;            /* [hidden] */
    const float *w_gate, *w_up;       /* [ffn_dim][hidden] */
    const float *w_down;              /* [hidden][ffn_dim] */
    uint32_t ffn_dim, reserved;
} wr_cuda_layer_desc;

typedef struct wr_cuda_model_desc {
    uint32_t n_layers, hidden, n_q_heads, n_kv_heads, head_dim, vocab;
    uint32_t n_rot_pairs;             /* as wr_cuda_kv_append */
    uint32_t max_rows;                /* rows one forward pass may carry (prefill chunk) */
    float rms_eps, rope_theta, attn_scale /* <= 0: 1/sqrt(head_dim) */, reserved;
    const float *embed, *lm_head, *final_norm;
    const wr_cuda_layer_desc *layers; /* n_layers entries */
} wr_cuda_model_desc;

/* Uploads every weight (one device allocation) and takes the row scratch; the
 * host copies are not referenced after the call returns. */
int  wr_cuda_model_create(wr_cuda_ctx *ctx, const wr_cuda_model_desc *desc, wr_cuda_model **out);
void wr_cuda_model_destroy(wr_cuda_model *m);
uint64_t wr_cuda_model_bytes(const wr_cuda_model *m);      /* device bytes held */
uint64_t wr_cuda_model_launches(const wr_cuda_model *m);   /* glue kernels launched so far */
/* host time, in ns, that the last forward pass spent enqueueing before it began to wait for the device */
uint64_t wr_cuda_model_last_enqueue_ns(const wr_cuda_model *m);

/* One forward pass over n_rows rows (decode: n_rows <= WR_CUDA_BATCH_MAX
 * sessions, one new token each; prefill: n_rows <= max_rows tokens of one
 * session), KV appended at `positions` as wr_cuda_decode_step /
 * wr_cuda_kv_append do — the caller commits the new length only when the call
 * returns 0.  A token id >= vocab is WR_CUDA_ERR_INVAL before anything runs
 * (session.c:413).  Results are written for rows [out_from, n_rows), all to
 * host memory, each pointer optional: hidden_out [n][hidden] (the residual
 * stream before the final norm), normed_out [n][hidden], logits_out[i] ->
 * [vocab] for row out_from+i (an entry may be NULL), argmax_out[i] = the first
 * maximum of that row's logits (the lowest id wins a tie, src/cli/wayrt.c:805).
 * Logits / arg-max for at most WR_CUDA_BATCH_MAX rows per call.  attn_tap_out,
 * when given, receives every layer's attention rows, [n_layers][n_rows][n_q*hd].
 * The call synchronises and reports a device-side give-up like every
 * host-buffer call.  One forward pass per model at a time (serialised inside). */
int wr_cuda_model_forward(wr_cuda_ctx *ctx, wr_cuda_model *m, int mode, uint32_t n_rows,
                          wr_cuda_kv *const *kv, const uint32_t *positions,
                          const uint32_t *tokens, uint32_t out_from, float *hidden_out,
                          float *normed_out, float *const *logits_out, uint32_t *argmax_out,
                          float *attn_tap_out);

/* ---- models whose layers differ ------------------------------------------- */

/* A model put together from mixers: every layer names its own mixer (softmax
 * attention, plain or differential; attention over a latent; selective scan) and
 * feed-forward (dense or a mixture of experts) with sizes of its own, a run list says in which order the layers are applied (a layer
 * may run several times with the same weights; each run keeps a cache or state
 * of its own).  It is a wr_cuda_model like the one above: created from host
 * pointers, stepped by wr_cuda_model_forward, destroyed by
 * wr_cuda_model_destroy; its sessions come from wr_cuda_model_kv_create.  (No
 * reference counterpart: the reference's decode body knows one layer shape per
 * architecture, src/core/session.c:405-568.)
 *
 * Tensors are host pointers with their element type (WR_CUDA_F32 or
 * WR_CUDA_BF16); a projection is [out][in] as everywhere in this header.
 * `compute` chooses the arithmetic: WR_CUDA_F32 keeps weights, activations and
 * K/V rows in 32 bits; WR_CUDA_BF16 keeps weights in BF16, runs the matrix
 * products of more than WR_CUDA_BATCH_MAX rows on BF16 activations with 32-bit
 * accumulation, and keeps K/V rows in F16 (rounded to nearest).  In both the
 * residual stream, norms, softmax and recurrences are 32-bit. */
typedef struct wr_cuda_tensor {
    const void *data;                 /* NULL: the layer does not have it */
    uint32_t dtype, reserved;
} wr_cuda_tensor;

#define WR_CUDA_MIXER_ATTENTION 1
#define WR_CUDA_MIXER_MAMBA1    2
#define WR_CUDA_MIXER_LATENT    3
#define WR_CUDA_FFN_NONE        0
#define WR_CUDA_FFN_POLYNORM    1
#define WR_CUDA_FFN_SWIGLU      2     /* w_down(silu(w_gate_up h) * (w_up h)) */
#define WR_CUDA_FFN_MOE         3     /* a mixture of experts (below) */
#define WR_CUDA_NORM_RMS        0
#define WR_CUDA_NORM_LAYER      1     /* the mean is taken off first */
#define WR_CUDA_POS_NONE        0
#define WR_CUDA_POS_SINUSOIDAL  1     /* added to the embedding: sin, cos of p * base^(-2i/width) interleaved */

typedef struct wr_cuda_mixed_layer {
    uint32_t mixer, ffn;
    uint32_t parallel, reserved0;     /* 1: the feed-forward reads norm1's output too and there is no norm2 */
    wr_cuda_tensor norm1, norm2;      /* [width]; norm2 only with a feed-forward of its own input */
    wr_cuda_tensor shift;             /* [width]: mixer input h + (h_before - h) * shift, or absent */

    /* WR_CUDA_MIXER_ATTENTION.  n_maps = 2 is differential attention: every
     * query head has two queries and every kv head two keys over one value, and
     * the head's output is (a1 - lambda a2) over its own root mean square (eps
     * diff_eps) times 1 - diff_init, lambda = exp(lq1.lk1) - exp(lq2.lk2) +
     * diff_init.  q rows are [head][map][k_dim], k rows [kv head][map][k_dim]. */
    uint32_t n_q_heads, n_kv_heads, n_maps, k_dim, v_dim;
    uint32_t q_temp_every;            /* > 0: q times 1 + coef ln(floor((p+1)/every) + 1) */
    float q_temp_coef, attn_scale, diff_init, diff_eps;
    wr_cuda_tensor wq, wk, wv, wo, bq, bk, bv;      /* biases optional */
    wr_cuda_tensor w_gate;            /* [n_q*v_dim][width]: heads times sigmoid(w_gate h), or absent */
    wr_cuda_tensor lq1, lk1, lq2, lk2;              /* [k_dim], n_maps = 2 */

    /* WR_CUDA_MIXER_MAMBA1: inner channels with `state` numbers each, a causal
     * convolution of `taps` taps, step sizes through rank dt_rank. */
    uint32_t inner, state, dt_rank, taps;
    wr_cuda_tensor w_in, conv, conv_b, w_x, w_dt, dt_b, a_log, d, w_out;

    /* WR_CUDA_FFN_POLYNORM: down(a N(z) + b N(z^2) + c N(z^3) + e), z = up h,
     * N = over its own root mean square (eps ffn_eps); act = {a, b, c, e}. */
    uint32_t ffn_dim;
    float ffn_eps;
    wr_cuda_tensor w_up, w_down, act;

    /* WR_CUDA_MIXER_LATENT: n_q_heads heads whose keys and values are linear in a
     * row of kv_rank numbers that all heads share, the only thing kept per token
     * besides one key part of rot_dim numbers with rotary positions (pairs i and
     * i + rot_dim/2, angle p * rope_base^(-2i/rot_dim)).  q = w_uq norm(w_dq h), per
     * head [k_dim | rot_dim rotated]; w_dkv h = [kv_rank, RMS-normed | rot_dim];
     * score = attn_scale (q . w_uk c + q_rot . k_rot), value = w_uv c.  kv_from = 1 +
     * j: the layer has no w_dkv and reads the rows that the latest run of layer j
     * before it has left; 0: its own. */
    uint32_t rot_dim, q_rank, kv_rank, kv_from;
    double rope_base;
    float latent_eps;
    uint32_t reserved1;
    wr_cuda_tensor w_dq, dq_norm, w_uq, w_dkv, dkv_norm, w_uk, w_uv;       /* and wo */

    /* WR_CUDA_FFN_SWIGLU: w_gate_up [ffn_dim][width], w_up, w_down.
     * WR_CUDA_FFN_MOE: of n_experts the top_k with the largest logits (router h +
     * router_b), weighted by the softmax over theirs; an expert of ffn_dim is
     * down(g sigmoid(moe_alpha g) (u + 1)), g = min(gate h, moe_limit), u = up h
     * within +-moe_limit.  experts: {gate, up, down} of every expert. */
    uint32_t n_experts, top_k;
    float moe_alpha, moe_limit;
    wr_cuda_tensor w_gate_up, router, router_b;
    const wr_cuda_tensor *experts;
} wr_cuda_mixed_layer;

typedef struct wr_cuda_mixed_desc {
    uint32_t compute;                 /* WR_CUDA_F32 or WR_CUDA_BF16 */
    uint32_t width, vocab, n_layers, n_runs;
    uint32_t max_rows;                /* rows one forward pass may carry (prefill chunk) */
    uint32_t norm_groups;             /* RMS norm over this many equal parts of the row */
    uint32_t position;                /* WR_CUDA_POS_* */
    float norm_eps, position_base;
    uint32_t norm;                    /* WR_CUDA_NORM_*, of norm1, norm2 and final_norm */
    float embed_scale, residual_mult; /* factor on embedding rows; on what a sublayer adds to the residual */
    uint32_t reserved;
    const uint32_t *runs;             /* n_runs layer indices, in the order they are applied */
    wr_cuda_tensor embed, head, final_norm;
    const wr_cuda_mixed_layer *layers;
} wr_cuda_mixed_desc;

int  wr_cuda_model_create_mixed(wr_cuda_ctx *ctx, const wr_cuda_mixed_desc *desc, wr_cuda_model **out);

/* An empty session for a model of either kind, for up to max_ctx tokens.  With
 * a mixed model wr_cuda_model_forward takes a step at the position the session
 * stands at, at the one before its last step again (that step is then undone),
 * or at 0 (the session starts over); any other position is WR_CUDA_ERR_STATE. */
int  wr_cuda_model_kv_create(wr_cuda_ctx *ctx, wr_cuda_model *m, uint32_t max_ctx, wr_cuda_kv **out);

/* wr_cuda_model_forward on a mixed model differs in three points: logits_out
 * may name any number of rows (NULL entries are skipped, only the named rows
 * reach the head), argmax_out still at most WR_CUDA_BATCH_MAX; attn_tap_out must
 * be NULL; and hidden_tap, when set with the call below, receives the residual
 * rows after every layer run of the following calls, [n_runs][n_rows][width]
 * (host memory; NULL turns it off). */
int  wr_cuda_model_set_hidden_tap(wr_cuda_model *m, float *hidden_tap);

#ifdef __cplusplus
}
#endif
#endif
