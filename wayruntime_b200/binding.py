"""ctypes mirror of include/wr_cuda.h.

Argument meaning and error behaviour are the C-ABI's: every call returns a
``wr_status`` value, and a negative one is raised as :class:`WrCudaError`
carrying that code.  Buffers may be numpy arrays or CPU torch tensors (host
memory: the call copies and synchronises) or CUDA torch tensors (device
memory: the call only enqueues on the context's stream).
"""
from __future__ import annotations

import ctypes as C
import os

import numpy as np

_PKG = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_PKG, "lib", "libwr_cuda.so")

MEM_HOST, MEM_DEVICE = 0, 1
F32, F16, BF16 = 0, 1, 2
APPEND_ROPE = 1
TRIPLE_PAD = 4
BATCH_MAX = 16

_STATUS = {
    0: "WR_OK", -3: "WR_ERR_UNSUPPORTED", -4: "WR_ERR_INVAL", -5: "WR_ERR_NOMEM",
    -6: "WR_ERR_CTX_FULL", -7: "WR_ERR_STATE", -8: "WR_ERR_LIMIT", -10: "WR_ERR_INTERNAL",
}

EXPORTS = [
    "wr_cuda_device_check", "wr_cuda_ctx_create", "wr_cuda_ctx_destroy", "wr_cuda_ctx_sync",
    "wr_cuda_ctx_stream", "wr_cuda_ctx_set_attn_max_seq", "wr_cuda_ctx_set_wait_limit",
    "wr_cuda_ctx_last_device_error",
    "wr_cuda_ctx_launch_count", "wr_cuda_host_alloc", "wr_cuda_host_free",
    "wr_cuda_kv_create", "wr_cuda_kv_destroy", "wr_cuda_kv_max_ctx", "wr_cuda_kv_write_rows",
    "wr_cuda_kv_read_rows", "wr_cuda_kv_append", "wr_cuda_attn_decode", "wr_cuda_attn_prefill",
    "wr_cuda_attn_decode_partial", "wr_cuda_attn_combine", "wr_cuda_decode_step",
    "wr_cuda_attn_decode_static",
    "wr_cuda_xchg_create", "wr_cuda_xchg_handle", "wr_cuda_xchg_connect", "wr_cuda_xchg_connect_local",
    "wr_cuda_xchg_destroy",
    "wr_cuda_attn_exchange_combine", "wr_cuda_attn_decode_exchange",
    "wr_cuda_model_create", "wr_cuda_model_destroy", "wr_cuda_model_bytes", "wr_cuda_model_launches", "wr_cuda_model_last_enqueue_ns",
    "wr_cuda_model_forward", "wr_cuda_kv_create_layout", "wr_cuda_model_create_mixed", "wr_cuda_model_kv_create",
    "wr_cuda_model_set_hidden_tap",
]


def status_name(rc: int) -> str:
    return _STATUS.get(rc, f"wr_status({rc})")


class WrCudaError(RuntimeError):
    def __init__(self, rc: int, what: str):
        super().__init__(f"{what}: {status_name(rc)}")
        self.status = rc


class LayerDesc(C.Structure):
    """wr_cuda_layer_desc (include/wr_cuda.h)."""
    _fields_ = [(n, C.c_void_p) for n in ("attn_norm", "wq", "wk", "wv", "q_norm", "k_norm", "wo",
                                          "ffn_norm", "w_gate", "w_up", "w_down")] + \
               [("ffn_dim", C.c_uint32), ("reserved", C.c_uint32)]


class ModelDesc(C.Structure):
    """wr_cuda_model_desc (include/wr_cuda.h)."""
    _fields_ = [(n, C.c_uint32) for n in ("n_layers", "hidden", "n_q_heads", "n_kv_heads", "head_dim",
                                          "vocab", "n_rot_pairs", "max_rows")] + \
               [(n, C.c_float) for n in ("rms_eps", "rope_theta", "attn_scale", "reserved")] + \
               [("embed", C.c_void_p), ("lm_head", C.c_void_p), ("final_norm", C.c_void_p),
                ("layers", C.POINTER(LayerDesc))]


class CacheLayer(C.Structure):
    """wr_cuda_cache_layer (include/wr_cuda.h)."""
    _fields_ = [(n, C.c_uint32) for n in ("n_kv_heads", "k_dim", "v_dim", "elem")] + [("state_bytes", C.c_uint64)]


class Tensor(C.Structure):
    """wr_cuda_tensor (include/wr_cuda.h)."""
    _fields_ = [("data", C.c_void_p), ("dtype", C.c_uint32), ("reserved", C.c_uint32)]


MIXER_ATTENTION, MIXER_MAMBA1, MIXER_LATENT = 1, 2, 3
FFN_NONE, FFN_POLYNORM, FFN_SWIGLU, FFN_MOE = 0, 1, 2, 3
NORM_RMS, NORM_LAYER = 0, 1
POS_NONE, POS_SINUSOIDAL = 0, 1


class MixedLayerDesc(C.Structure):
    """wr_cuda_mixed_layer (include/wr_cuda.h)."""
    TENSORS = ("norm1", "norm2", "shift", "wq", "wk", "wv", "wo", "bq", "bk", "bv", "w_gate", "lq1", "lk1", "lq2", "lk2",
               "w_in", "conv", "conv_b", "w_x", "w_dt", "dt_b", "a_log", "d", "w_out", "w_up", "w_down", "act",
               "w_dq", "dq_norm", "w_uq", "w_dkv", "dkv_norm", "w_uk", "w_uv", "w_gate_up", "router", "router_b")
    _fields_ = [(n, C.c_uint32) for n in ("mixer", "ffn", "parallel", "reserved0")] + [(n, Tensor) for n in ("norm1", "norm2", "shift")] + \
               [(n, C.c_uint32) for n in ("n_q_heads", "n_kv_heads", "n_maps", "k_dim", "v_dim", "q_temp_every")] + \
               [(n, C.c_float) for n in ("q_temp_coef", "attn_scale", "diff_init", "diff_eps")] + \
               [(n, Tensor) for n in ("wq", "wk", "wv", "wo", "bq", "bk", "bv", "w_gate", "lq1", "lk1", "lq2", "lk2")] + \
               [(n, C.c_uint32) for n in ("inner", "state", "dt_rank", "taps")] + \
               [(n, Tensor) for n in ("w_in", "conv", "conv_b", "w_x", "w_dt", "dt_b", "a_log", "d", "w_out")] + \
               [("ffn_dim", C.c_uint32), ("ffn_eps", C.c_float)] + [(n, Tensor) for n in ("w_up", "w_down", "act")] + \
               [(n, C.c_uint32) for n in ("rot_dim", "q_rank", "kv_rank", "kv_from")] + \
               [("rope_base", C.c_double), ("latent_eps", C.c_float), ("reserved1", C.c_uint32)] + \
               [(n, Tensor) for n in ("w_dq", "dq_norm", "w_uq", "w_dkv", "dkv_norm", "w_uk", "w_uv")] + \
               [("n_experts", C.c_uint32), ("top_k", C.c_uint32), ("moe_alpha", C.c_float), ("moe_limit", C.c_float)] + \
               [(n, Tensor) for n in ("w_gate_up", "router", "router_b")] + [("experts", C.POINTER(Tensor))]


class MixedDesc(C.Structure):
    """wr_cuda_mixed_desc (include/wr_cuda.h)."""
    _fields_ = [(n, C.c_uint32) for n in ("compute", "width", "vocab", "n_layers", "n_runs", "max_rows", "norm_groups",
                                          "position")] + \
               [("norm_eps", C.c_float), ("position_base", C.c_float), ("norm", C.c_uint32), ("embed_scale", C.c_float),
                ("residual_mult", C.c_float), ("reserved", C.c_uint32), ("runs", C.POINTER(C.c_uint32))] + \
               [(n, Tensor) for n in ("embed", "head", "final_norm")] + [("layers", C.POINTER(MixedLayerDesc))]


_lib = None


def load_library():
    """Load libwr_cuda.so; raises if it was never built (no fallback exists)."""
    global _lib
    if _lib is not None:
        return _lib
    if not os.path.exists(LIB_PATH):
        raise RuntimeError(
            f"{LIB_PATH} is missing: build it with `python -c 'import __graft_entry__ as g; "
            "g.build()'` (needs nvcc); wayruntime_b200 has no CPU path")
    lib = C.CDLL(LIB_PATH)
    vp, u32, i32, f32 = C.c_void_p, C.c_uint32, C.c_int, C.c_float
    sig = {
        "wr_cuda_device_check": (i32, [i32]),
        "wr_cuda_ctx_create": (i32, [i32, C.POINTER(vp)]),
        "wr_cuda_ctx_destroy": (None, [vp]),
        "wr_cuda_ctx_sync": (i32, [vp]),
        "wr_cuda_ctx_stream": (vp, [vp]),
        "wr_cuda_ctx_set_attn_max_seq": (i32, [vp, u32]),
        "wr_cuda_ctx_set_wait_limit": (i32, [vp, C.c_int64]),
        "wr_cuda_ctx_last_device_error": (i32, [vp]),
        "wr_cuda_ctx_launch_count": (C.c_uint64, [vp]),
        "wr_cuda_host_alloc": (i32, [vp, C.c_uint64, C.POINTER(vp)]),
        "wr_cuda_host_free": (None, [vp, vp]),
        "wr_cuda_kv_create": (i32, [vp, u32, u32, u32, u32, C.POINTER(vp)]),
        "wr_cuda_kv_destroy": (None, [vp]),
        "wr_cuda_kv_max_ctx": (u32, [vp]),
        "wr_cuda_kv_write_rows": (i32, [vp, vp, u32, i32, u32, u32, vp, i32]),
        "wr_cuda_kv_read_rows": (i32, [vp, vp, u32, i32, u32, u32, vp, i32]),
        "wr_cuda_kv_append": (i32, [vp, u32, C.POINTER(vp), u32, C.POINTER(u32), u32, vp, vp, vp,
                                    u32, f32, u32, u32, i32]),
        "wr_cuda_attn_decode": (i32, [vp, u32, C.POINTER(vp), u32, C.POINTER(u32), vp, vp, u32,
                                      f32, u32, i32]),
        "wr_cuda_attn_prefill": (i32, [vp, vp, u32, u32, u32, vp, i32, vp, u32, f32, u32, i32]),
        "wr_cuda_attn_decode_partial": (i32, [vp, u32, C.POINTER(vp), u32, C.POINTER(u32), vp, vp,
                                              u32, f32, i32]),
        "wr_cuda_attn_combine": (i32, [vp, u32, u32, u32, vp, vp, i32]),
        "wr_cuda_decode_step": (i32, [vp, u32, C.POINTER(vp), u32, C.POINTER(u32), vp, vp, vp, vp,
                                      u32, f32, u32, u32, f32, u32, i32]),
        "wr_cuda_attn_decode_static": (i32, [vp, u32, C.POINTER(vp), u32, C.POINTER(u32), vp, vp,
                                             u32, f32, u32]),
        "wr_cuda_xchg_create": (i32, [vp, u32, u32, u32, u32, C.POINTER(vp)]),
        "wr_cuda_xchg_handle": (i32, [vp, vp]),
        "wr_cuda_xchg_connect": (i32, [vp, vp]),
        "wr_cuda_xchg_connect_local": (i32, [vp, C.POINTER(vp)]),
        "wr_cuda_xchg_destroy": (None, [vp]),
        "wr_cuda_attn_exchange_combine": (i32, [vp, vp, u32, vp, vp]),
        "wr_cuda_attn_decode_exchange": (i32, [vp, vp, u32, C.POINTER(vp), u32, C.POINTER(u32), vp, vp, u32, f32]),
        "wr_cuda_model_create": (i32, [vp, C.POINTER(ModelDesc), C.POINTER(vp)]),
        "wr_cuda_model_destroy": (None, [vp]),
        "wr_cuda_model_bytes": (C.c_uint64, [vp]),
        "wr_cuda_model_launches": (C.c_uint64, [vp]),
        "wr_cuda_model_last_enqueue_ns": (C.c_uint64, [vp]),
        "wr_cuda_kv_create_layout": (i32, [vp, u32, C.POINTER(CacheLayer), u32, C.POINTER(vp)]),
        "wr_cuda_model_create_mixed": (i32, [vp, C.POINTER(MixedDesc), C.POINTER(vp)]),
        "wr_cuda_model_kv_create": (i32, [vp, vp, u32, C.POINTER(vp)]),
        "wr_cuda_model_set_hidden_tap": (i32, [vp, vp]),
        "wr_cuda_model_forward": (i32, [vp, vp, i32, u32, C.POINTER(vp), C.POINTER(u32), C.POINTER(u32), u32,
                                        vp, vp, C.POINTER(vp), C.POINTER(u32), vp]),
    }
    for name, (res, args) in sig.items():
        fn = getattr(lib, name)
        fn.restype = res
        fn.argtypes = args
    _lib = lib
    return lib


def device_check(device: int = 0) -> int:
    """wr_status: 0 when `device` is an sm_100 GPU, WR_ERR_UNSUPPORTED otherwise."""
    return int(load_library().wr_cuda_device_check(device))


def _buf(x):
    """(address, mem kind, keep-alive) of a numpy array / torch tensor."""
    if x is None:
        return None, None, None
    if isinstance(x, np.ndarray):
        if not x.flags["C_CONTIGUOUS"]:
            raise ValueError("buffers must be C-contiguous")
        return x.ctypes.data, MEM_HOST, x
    if hasattr(x, "data_ptr"):
        if not x.is_contiguous():
            raise ValueError("buffers must be contiguous")
        return x.data_ptr(), (MEM_DEVICE if x.is_cuda else MEM_HOST), x
    raise TypeError(f"unsupported buffer {type(x)}")


def _same_mem(*kinds):
    ks = {k for k in kinds if k is not None}
    if len(ks) != 1:
        raise ValueError("all buffers of one call must live on the same side (host or device)")
    return ks.pop()


def _check(rc, what):
    if rc != 0:
        raise WrCudaError(int(rc), what)


class Context:
    """One device, one stream, one page pool (wr_cuda_ctx)."""

    def __init__(self, device: int = 0, attn_max_seq: int | None = None):
        self._lib = load_library()
        h = C.c_void_p()
        _check(self._lib.wr_cuda_ctx_create(device, C.byref(h)), "wr_cuda_ctx_create")
        self._h = h
        self.device = device
        if attn_max_seq is not None:
            self.set_attn_max_seq(attn_max_seq)

    def close(self):
        if getattr(self, "_h", None):
            self._lib.wr_cuda_ctx_destroy(self._h)
            self._h = None

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass

    def sync(self):
        _check(self._lib.wr_cuda_ctx_sync(self._h), "wr_cuda_ctx_sync")

    @property
    def stream(self) -> int:
        return int(self._lib.wr_cuda_ctx_stream(self._h) or 0)

    @property
    def launch_count(self) -> int:
        return int(self._lib.wr_cuda_ctx_launch_count(self._h))

    def set_attn_max_seq(self, n: int):
        _check(self._lib.wr_cuda_ctx_set_attn_max_seq(self._h, n), "wr_cuda_ctx_set_attn_max_seq")

    @property
    def last_device_error(self) -> int:
        """Error word of the last device-side give-up that was reported (0: none)."""
        return int(self._lib.wr_cuda_ctx_last_device_error(self._h))

    def set_wait_limit(self, cycles: int):
        """SM clock cycles after which a device-side wait gives up (default about 2 s)."""
        _check(self._lib.wr_cuda_ctx_set_wait_limit(self._h, int(cycles)), "wr_cuda_ctx_set_wait_limit")

    def kv_create(self, n_layers, n_kv_heads, head_dim, max_ctx) -> "KVCache":
        return KVCache(self, n_layers, n_kv_heads, head_dim, max_ctx)

    # ---- the hot path -------------------------------------------------
    @staticmethod
    def _handles(kvs):
        if isinstance(kvs, Batch):
            return kvs.handles
        return (C.c_void_p * len(kvs))(*[k._h for k in kvs])

    @staticmethod
    def _u32s(vals):
        if isinstance(vals, C.Array):
            return vals
        return (C.c_uint32 * len(vals))(*[int(v) for v in vals])

    def decode_step(self, kvs, layer, positions, q, k_rows, v_rows, out, n_q_heads, theta=10000.0,
                    n_rot_pairs=0, rope=True, scale=0.0, window=0):
        qp, qm, _q = _buf(q)
        kp, km, _k = _buf(k_rows)
        vp, vm, _v = _buf(v_rows)
        op, om, _o = _buf(out)
        mem = _same_mem(qm, km, vm, om)
        rc = self._lib.wr_cuda_decode_step(self._h, len(kvs), self._handles(kvs), layer,
                                           self._u32s(positions), qp, kp, vp, op, n_q_heads, theta,
                                           n_rot_pairs, APPEND_ROPE if rope else 0, scale, window,
                                           mem)
        _check(rc, "wr_cuda_decode_step")

    def prepared_decode_step(self, kvs, positions, q, k_rows, v_rows, out, n_q_heads, theta=10000.0,
                             n_rot_pairs=0, rope=True, scale=0.0, window=0):
        """wr_cuda_decode_step with everything but the layer resolved once: returns `step(layer)`.
        For a serving loop that steps the same sessions and buffers over and over — the C caller's
        situation, where the arguments are pointers it already holds — so that a call costs the
        library's work and not the marshalling of its arguments.  positions: a list (copied once) or
        a ctypes array from Batch.u32 that the caller updates in place between steps."""
        qp, qm, _q = _buf(q)
        kp, km, _k = _buf(k_rows)
        vp, vm, _v = _buf(v_rows)
        op, om, _o = _buf(out)
        mem = _same_mem(qm, km, vm, om)
        handles, pos = self._handles(kvs), self._u32s(positions)
        n = len(kvs)
        fn, ctx_h = self._lib.wr_cuda_decode_step, self._h
        flags = APPEND_ROPE if rope else 0
        keep = (_q, _k, _v, _o, handles, pos)

        def step(layer, _keep=keep):
            rc = fn(ctx_h, n, handles, layer, pos, qp, kp, vp, op, n_q_heads, theta, n_rot_pairs, flags, scale,
                    window, mem)
            if rc != 0:
                raise WrCudaError(int(rc), "wr_cuda_decode_step")

        return step

    def kv_append(self, kvs, layer, positions, k_rows, v_rows, q_rows=None, n_q_heads=0,
                  theta=10000.0, n_rot_pairs=0, rope=True, n_tokens=1):
        kp, km, _k = _buf(k_rows)
        vp, vm, _v = _buf(v_rows)
        qp, qm, _q = _buf(q_rows)
        mem = _same_mem(km, vm, qm)
        pos = self._u32s(positions)
        rc = self._lib.wr_cuda_kv_append(self._h, len(kvs), self._handles(kvs), layer, pos,
                                         n_tokens, kp, vp, qp, n_q_heads, theta, n_rot_pairs,
                                         APPEND_ROPE if rope else 0, mem)
        _check(rc, "wr_cuda_kv_append")

    def attn_decode(self, kvs, layer, seq_lens, q, out, n_q_heads, scale=0.0, window=0):
        qp, qm, _q = _buf(q)
        op, om, _o = _buf(out)
        mem = _same_mem(qm, om)
        lens = self._u32s(seq_lens)
        rc = self._lib.wr_cuda_attn_decode(self._h, len(kvs), self._handles(kvs), layer, lens, qp,
                                           op, n_q_heads, scale, window, mem)
        _check(rc, "wr_cuda_attn_decode")

    def attn_decode_static(self, kvs, layer, seq_lens, q, out, n_q_heads, scale=0.0, window=0):
        """wr_cuda_attn_decode_static: the decode kernel over the library's fixed
        scratch array, for callers that may not allocate.  q and out must be
        device buffers; oversize calls raise WR_ERR_LIMIT."""
        qp, qm, _q = _buf(q)
        op, om, _o = _buf(out)
        if qm != MEM_DEVICE or om != MEM_DEVICE:
            raise ValueError("wr_cuda_attn_decode_static takes device buffers only")
        rc = self._lib.wr_cuda_attn_decode_static(self._h, len(kvs), self._handles(kvs), layer,
                                                  self._u32s(seq_lens), qp, op, n_q_heads, scale,
                                                  window)
        _check(rc, "wr_cuda_attn_decode_static")

    def attn_decode_partial(self, kvs, layer, seq_lens, q, triples, n_q_heads, scale=0.0):
        qp, qm, _q = _buf(q)
        tp, tm, _t = _buf(triples)
        mem = _same_mem(qm, tm)
        lens = self._u32s(seq_lens)
        rc = self._lib.wr_cuda_attn_decode_partial(self._h, len(kvs), self._handles(kvs), layer,
                                                   lens, qp, tp, n_q_heads, scale, mem)
        _check(rc, "wr_cuda_attn_decode_partial")

    def attn_combine(self, n_shards, n_rows, head_dim, triples, out):
        tp, tm, _t = _buf(triples)
        op, om, _o = _buf(out)
        mem = _same_mem(tm, om)
        rc = self._lib.wr_cuda_attn_combine(self._h, n_shards, n_rows, head_dim, tp, op, mem)
        _check(rc, "wr_cuda_attn_combine")

    def attn_prefill(self, kv, layer, p0, n, q, out, n_q_heads, scale=0.0, window=0):
        qp, qm, qa = _buf(q)
        op, om, _o = _buf(out)
        mem = _same_mem(qm, om)
        if isinstance(qa, np.ndarray):
            q_dtype = F32 if qa.dtype == np.float32 else F16
        else:
            q_dtype = F32 if qa.element_size() == 4 else F16
        rc = self._lib.wr_cuda_attn_prefill(self._h, kv._h, layer, p0, n, qp, q_dtype, op,
                                            n_q_heads, scale, window, mem)
        _check(rc, "wr_cuda_attn_prefill")


XCHG_HANDLE_BYTES = 64


class Exchange:
    """Peer buffers for the fused all-gather + merge of split-KV triples
    (wr_cuda_xchg): create on every rank, pass everybody's `handle` (rank order)
    to `connect`, then call `combine` once per step on every rank."""

    def __init__(self, ctx: "Context", world: int, rank: int, max_rows: int, head_dim: int):
        self._ctx = ctx
        self._lib = ctx._lib
        self.world, self.rank = world, rank
        h = C.c_void_p()
        _check(self._lib.wr_cuda_xchg_create(ctx._h, world, rank, max_rows, head_dim, C.byref(h)),
               "wr_cuda_xchg_create")
        self._h = h

    @property
    def handle(self) -> bytes:
        buf = C.create_string_buffer(XCHG_HANDLE_BYTES)
        _check(self._lib.wr_cuda_xchg_handle(self._h, buf), "wr_cuda_xchg_handle")
        return buf.raw

    def connect(self, handles) -> None:
        blob = b"".join(handles)
        if len(blob) != self.world * XCHG_HANDLE_BYTES:
            raise ValueError("one 64-byte handle per rank, in rank order")
        _check(self._lib.wr_cuda_xchg_connect(self._h, C.c_char_p(blob)), "wr_cuda_xchg_connect")

    @staticmethod
    def connect_local(objs) -> None:
        """Connect exchange objects that live in this process (rank order)."""
        arr = (C.c_void_p * len(objs))(*[o._h for o in objs])
        for o in objs:
            _check(o._lib.wr_cuda_xchg_connect_local(o._h, arr), "wr_cuda_xchg_connect_local")

    def combine(self, n_rows: int, triples, out) -> None:
        tp, tm, _t = _buf(triples)
        op, om, _o = _buf(out)
        if tm != MEM_DEVICE or om != MEM_DEVICE:
            raise ValueError("wr_cuda_attn_exchange_combine takes device buffers only")
        _check(self._lib.wr_cuda_attn_exchange_combine(self._ctx._h, self._h, n_rows, tp, op),
               "wr_cuda_attn_exchange_combine")

    def decode(self, kvs, layer, seq_lens, q, out, n_q_heads, scale=0.0) -> None:
        """wr_cuda_attn_decode_exchange: partial attention over this rank's keys with the
        exchange and the merge fused in (device buffers)."""
        qp, qm, _q = _buf(q)
        op, om, _o = _buf(out)
        if qm != MEM_DEVICE or om != MEM_DEVICE:
            raise ValueError("wr_cuda_attn_decode_exchange takes device buffers only")
        _check(self._lib.wr_cuda_attn_decode_exchange(self._ctx._h, self._h, len(kvs), Context._handles(kvs), layer,
                                                      Context._u32s(seq_lens), qp, op, n_q_heads, scale),
               "wr_cuda_attn_decode_exchange")

    def close(self) -> None:
        if self._h:
            self._lib.wr_cuda_xchg_destroy(self._h)
            self._h = None


class DeviceModel:
    """wr_cuda_model: a model's F32 weights mirrored on the device and the layer
    stack around attention run there.  `weights` maps names to C-contiguous
    float32 numpy arrays in GGML layout (a [in -> out] projection is [out][in]):
    embed, lm_head (may be the same array), final_norm, and per layer i
    `l{i}.attn_norm|wq|wk|wv|q_norm|k_norm|wo|ffn_norm|w_gate|w_up|w_down`."""

    FWD_DECODE, FWD_PREFILL = 0, 1

    def __init__(self, ctx: "Context", weights: dict, *, n_layers, hidden, n_q_heads, n_kv_heads, head_dim,
                 vocab, ffn, rms_eps=1e-6, rope_theta=10000.0, n_rot_pairs=0, attn_scale=0.0, max_rows=256):
        self._ctx, self._lib = ctx, ctx._lib
        self.vocab, self.hidden, self.n_layers, self.max_rows = vocab, hidden, n_layers, max_rows
        self.n_q, self.hd = n_q_heads, head_dim

        def ptr(name, optional=False):
            a = weights.get(name)
            if a is None:
                if optional:
                    return None
                raise KeyError(name)
            if a.dtype != np.float32 or not a.flags["C_CONTIGUOUS"]:
                raise ValueError(f"{name}: C-contiguous float32 expected")
            return a.ctypes.data

        layers = (LayerDesc * n_layers)()
        for i in range(n_layers):
            for f in ("attn_norm", "wq", "wk", "wv", "wo", "ffn_norm", "w_gate", "w_up", "w_down"):
                setattr(layers[i], f, ptr(f"l{i}.{f}"))
            layers[i].q_norm = ptr(f"l{i}.q_norm", optional=True)
            layers[i].k_norm = ptr(f"l{i}.k_norm", optional=True)
            layers[i].ffn_dim = ffn[i] if isinstance(ffn, (list, tuple)) else ffn
        d = ModelDesc(n_layers=n_layers, hidden=hidden, n_q_heads=n_q_heads, n_kv_heads=n_kv_heads,
                      head_dim=head_dim, vocab=vocab, n_rot_pairs=n_rot_pairs, max_rows=max_rows,
                      rms_eps=rms_eps, rope_theta=rope_theta, attn_scale=attn_scale,
                      embed=ptr("embed"), lm_head=ptr("lm_head"), final_norm=ptr("final_norm"), layers=layers)
        h = C.c_void_p()
        _check(self._lib.wr_cuda_model_create(ctx._h, C.byref(d), C.byref(h)), "wr_cuda_model_create")
        self._h = h

    def close(self):
        if self._h:
            self._lib.wr_cuda_model_destroy(self._h)
            self._h = None

    @property
    def device_bytes(self) -> int:
        return int(self._lib.wr_cuda_model_bytes(self._h))

    @property
    def launches(self) -> int:
        return int(self._lib.wr_cuda_model_launches(self._h))

    @property
    def last_enqueue_ms(self) -> float:
        """Host time the last forward pass spent enqueueing work, before waiting for the device."""
        return self._lib.wr_cuda_model_last_enqueue_ns(self._h) * 1e-6

    def kv_create(self, max_ctx: int) -> "KVCache":
        """An empty session of this model for up to max_ctx tokens."""
        h = C.c_void_p()
        _check(self._lib.wr_cuda_model_kv_create(self._ctx._h, self._h, max_ctx, C.byref(h)), "wr_cuda_model_kv_create")
        return KVCache._of_handle(self._ctx, h, max_ctx)

    def forward(self, mode, kvs, positions, tokens, out_from=0, *, hidden=False, normed=False, logits=False,
                argmax=False, attn_tap=False) -> dict:
        """One forward pass; returns the requested results for rows [out_from, n) as numpy arrays.
        logits may be a list of places among those rows (the others are skipped): the result then has
        one row per place, in the list's order."""
        n = len(tokens)
        n_out = n - out_from
        res = {}
        hid = np.empty((n_out, self.hidden), np.float32) if hidden else None
        nrm = np.empty((n_out, self.hidden), np.float32) if normed else None
        some = None if isinstance(logits, bool) else [int(i) for i in logits]
        logits = bool(some) if some is not None else logits
        lg = np.empty((len(some) if some is not None else n_out, self.vocab), np.float32) if logits else None
        am = (C.c_uint32 * max(n_out, 1))() if argmax else None
        tap = np.empty((self.n_layers, n, self.n_q * self.hd), np.float32) if attn_tap else None
        lptrs = None
        if logits:
            lptrs = (C.c_void_p * max(n_out, 1))()
            base, row = lg.ctypes.data, lg.strides[0]
            for j, i in enumerate(some if some is not None else range(n_out)):
                if not 0 <= i < n_out or lptrs[i]:
                    raise ValueError("places out of range or named twice")
                lptrs[i] = base + j * row
        _check(self._lib.wr_cuda_model_forward(
            self._ctx._h, self._h, mode, n, Context._handles(kvs), Context._u32s(positions),
            Context._u32s(tokens), out_from, hid.ctypes.data if hidden else None,
            nrm.ctypes.data if normed else None, lptrs, am, tap.ctypes.data if attn_tap else None),
            "wr_cuda_model_forward")
        if hidden: res["hidden"] = hid
        if normed: res["normed"] = nrm
        if logits: res["logits"] = lg
        if argmax: res["argmax"] = np.array([am[i] for i in range(n_out)], np.uint32)
        if attn_tap: res["attn"] = tap
        return res


class MixedModel(DeviceModel):
    """wr_cuda_model of the mixed kind (wr_cuda_model_create_mixed).  `layers` is a list of dicts with the
    scalar fields of wr_cuda_mixed_layer; `tensor(i, field)` returns layer i's array for a tensor field (or None;
    for "experts" the gate, up and down arrays of every expert, one after the other), and tensor(None, name) the
    model's embed, head and final_norm.  Arrays are float32, or uint16 holding
    bfloat16 bits."""

    def __init__(self, ctx: "Context", layers, runs, tensor, *, compute, width, vocab, norm_groups, norm_eps,
                 position=POS_NONE, position_base=10000.0, norm=NORM_RMS, embed_scale=1.0, residual_mult=1.0, max_rows=256):
        self._ctx, self._lib = ctx, ctx._lib
        self.vocab, self.hidden, self.n_layers, self.max_rows = vocab, width, len(runs), max_rows
        self.n_q = self.hd = 0
        keep = []

        def ref(a):
            if a is None:
                return Tensor()
            if a.dtype not in (np.float32, np.uint16):
                raise ValueError("float32, or bfloat16 bits in uint16, expected")
            a = np.ascontiguousarray(a)
            keep.append(a)
            return Tensor(a.ctypes.data, F32 if a.dtype == np.float32 else BF16, 0)

        arr = (MixedLayerDesc * len(layers))()
        for i, lay in enumerate(layers):
            for k, v in lay.items():
                setattr(arr[i], k, v)
            for k in MixedLayerDesc.TENSORS:
                setattr(arr[i], k, ref(tensor(i, k)))
            if lay.get("n_experts"):
                parts = [ref(a) for a in tensor(i, "experts")]
                arr[i].experts = (Tensor * len(parts))(*parts)
        d = MixedDesc(compute=compute, width=width, vocab=vocab, n_layers=len(layers), n_runs=len(runs),
                      max_rows=max_rows, norm_groups=norm_groups, position=position, norm_eps=norm_eps,
                      position_base=position_base, norm=norm, embed_scale=embed_scale, residual_mult=residual_mult, runs=(C.c_uint32 * len(runs))(*runs), embed=ref(tensor(None, "embed")),
                      head=ref(tensor(None, "head")), final_norm=ref(tensor(None, "final_norm")), layers=arr)
        h = C.c_void_p()
        _check(self._lib.wr_cuda_model_create_mixed(ctx._h, C.byref(d), C.byref(h)), "wr_cuda_model_create_mixed")
        self._h = h

    def set_hidden_tap(self, out):
        """Residual rows after every layer run of the following forward calls into `out`
        (float32 [runs, rows, width]; None turns it off)."""
        _check(self._lib.wr_cuda_model_set_hidden_tap(self._h, None if out is None else out.ctypes.data),
               "wr_cuda_model_set_hidden_tap")
        self._tap = out


class Batch:
    """A fixed list of sessions with its handle array built once (saves the
    per-call marshalling when the same batch steps many times)."""

    def __init__(self, kvs):
        self.kvs = list(kvs)
        self.handles = (C.c_void_p * len(self.kvs))(*[k._h for k in self.kvs])

    def __len__(self):
        return len(self.kvs)

    @staticmethod
    def u32(vals):
        return (C.c_uint32 * len(vals))(*[int(v) for v in vals])


class KVCache:
    """One session's paged F16 K/V cache (wr_cuda_kv)."""

    def __init__(self, ctx: Context, n_layers, n_kv_heads, head_dim, max_ctx):
        self._ctx = ctx
        self._lib = ctx._lib
        h = C.c_void_p()
        _check(self._lib.wr_cuda_kv_create(ctx._h, n_layers, n_kv_heads, head_dim, max_ctx,
                                           C.byref(h)), "wr_cuda_kv_create")
        self._h = h
        self.n_layers, self.n_kv_heads, self.head_dim, self.max_ctx = (
            n_layers, n_kv_heads, head_dim, max_ctx)

    @classmethod
    def _of_handle(cls, ctx, handle, max_ctx):
        kv = cls.__new__(cls)
        kv._ctx, kv._lib, kv._h, kv.max_ctx = ctx, ctx._lib, handle, max_ctx
        kv.n_layers = kv.n_kv_heads = kv.head_dim = None
        return kv

    def close(self):
        if getattr(self, "_h", None) and getattr(self._ctx, "_h", None):
            self._lib.wr_cuda_kv_destroy(self._h)
        self._h = None

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass

    def write_rows(self, layer, which, row0, rows):
        """rows: uint16/float16 [n, n_kv_heads, head_dim] in the reference's row layout."""
        p, mem, _a = _buf(rows)
        n = rows.shape[0]
        _check(self._lib.wr_cuda_kv_write_rows(self._ctx._h, self._h, layer, which, row0, n, p, mem),
               "wr_cuda_kv_write_rows")

    def read_rows(self, layer, which, row0, n):
        out = np.empty((n, self.n_kv_heads, self.head_dim), np.uint16)
        _check(self._lib.wr_cuda_kv_read_rows(self._ctx._h, self._h, layer, which, row0, n,
                                              out.ctypes.data, MEM_HOST), "wr_cuda_kv_read_rows")
        return out
