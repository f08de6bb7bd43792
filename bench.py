#!/usr/bin/env python
"""bench.py — batched decode attention (benchmark config 2) on N GPUs of one node.

    python bench.py [--gpus N] [--steps K] [--warmup W] [--impl reference]

Workload ("c2_batched_decode"): Llama-3-8B geometry, 16 sessions per GPU,
32 Q heads / 8 KV heads, head_dim 128, F32 Q ~N(0,1), F16 K/V caches ~N(0,1)
with seeded context lengths uniform in [1024, 4096].  One step = one layer-step
of the hot path for the batch: fused RoPE + KV append of the 16 new rows, then
decode attention of all sessions in one grid.  Steps rotate over 4 independent
layer caches (each larger than L2) so every step streams K/V from HBM.

With N GPUs the job is N x 16 sessions drawn from one seed and spread over the
GPUs by wayruntime_b200.placement.assign_sessions (even summed context length,
16 sessions each, no data-path collective).

Prints ONE JSON line (rank 0).  `value` is whole-job tokens/s with inputs
resident in HBM (median over back-to-back repetitions of the K-step region);
`e2e` is the same step driven through the C-ABI with pinned HOST buffers
(copies inside the timed region); `roofline` is the decode kernel's
algorithmic bytes over its own CUDA-event time; `cpu_baseline` is the
reference's CPU attention timed on this box's host cores (all threads, and
one thread).  The two multi-GPU sections (`kv_head_sharded`, `split_kv`) come
last in the line, each with its own parity figure against the CPU reference.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time

import numpy as np

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

N_SESS, HQ, HKV, HD = 16, 32, 8, 128
CTX_LO, CTX_HI = 1024, 4096
N_ROT_LAYERS = 4
THETA = 500000.0
SEED = 20261125
# dram__bytes_read.sum + dram__bytes_write.sum per launch from the committed ncu captures
# (profiles/): same seeded workloads as the ones timed here.
NCU_TRAFFIC_DECODE_C2 = 171_000_000      # algorithmic 165 429 248 B
NCU_TRAFFIC_PREFILL_C3 = 25_800_000      # operands are re-read from L2
METRIC = "batched_decode_attention_tokens_per_s"
UNIT = "tok/s"


MIN_TIMED_S = 0.2           # the K-step region is repeated until this much device time is covered


def session_lengths(rank: int, world: int = 1) -> list[int]:
    """Context lengths of the 16 sessions GPU `rank` serves: the job's
    world x 16 seeded lengths, spread so that every GPU streams about the same
    number of cached keys per step."""
    from wayruntime_b200 import placement
    rng = np.random.Generator(np.random.Philox(SEED))
    all_lens = [int(x) for x in rng.integers(CTX_LO, CTX_HI + 1, size=N_SESS * world)]
    mine = placement.assign_sessions(all_lens, world, N_SESS)[rank]
    return [all_lens[i] for i in mine]


def r4(x):
    """Round for the JSON line (5 significant digits)."""
    return None if x is None else float(f"{float(x):.5g}")


def algorithmic_bytes(lens) -> int:
    """K+V of every cached row read once, plus Q in and O out (F32)."""
    kv = sum(lens) * HKV * HD * 2 * 2
    return kv + 2 * N_SESS * HQ * HD * 4


def measured_peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            return float(json.load(f)["hbm_gbs"]), "measured"
    return 6650.0, "fallback"


# ------------------------------------------------------------------ clocks

class ClockSampler:
    """Samples nvidia-smi SM clocks and throttle reasons while the timed region runs."""
    FIELDS = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
              "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_index: int):
        self.gpu = gpu_index
        self.rows: list[list[str]] = []
        self.proc = None
        self.thread = None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits",
                 "-lms", "50", "-i", str(self.gpu)],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.proc = None
            return
        self.thread = threading.Thread(target=self._read, daemon=True)
        self.thread.start()

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) >= 9:
                self.rows.append(parts)

    def stop(self) -> dict:
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        time.sleep(0.15)
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
        sm, smax, reasons = [], [], set()
        for r in self.rows:
            try:
                sm.append(float(r[1])), smax.append(float(r[2]))
            except ValueError:
                continue
            for name, val in zip(("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown",
                                  "sw_power_cap"), r[5:9]):
                if val.lower().startswith("active"):
                    reasons.add(name)
        return {"sm_mhz": float(np.median(sm)) if sm else None,
                "sm_max_mhz": max(smax) if smax else None,
                "samples": len(sm), "reasons": sorted(reasons)}


# ------------------------------------------------------------ CPU baseline

def cpu_checker():
    import oracle
    ref = oracle.reference()
    if ref is not None:
        return ref, "reference"
    return oracle.restatement(), "port"


def cpu_decode_once(chk, q, ks, vs, threads):
    t0 = time.perf_counter()
    rc, out = chk.decode_batch(q, ks, vs, threads=threads)
    dt = time.perf_counter() - t0
    if rc != 0:
        raise RuntimeError(f"CPU reference attention returned {rc}")
    return dt, out


def host_inputs(rank: int, world: int = 1):
    """Seeded host copies of the workload (used by the CPU arm): q F32,
    k/v uint16 rows per session."""
    lens = session_lengths(rank, world)
    rng = np.random.Generator(np.random.Philox(SEED + 1000 + rank))
    q = rng.standard_normal((N_SESS, HQ, HD), dtype=np.float32)
    ks = [rng.standard_normal((n, HKV, HD), dtype=np.float32).astype(np.float16).view(np.uint16)
          for n in lens]
    vs = [rng.standard_normal((n, HKV, HD), dtype=np.float32).astype(np.float16).view(np.uint16)
          for n in lens]
    return lens, q, ks, vs


def run_reference_arm(args):
    """The reference's own CPU attention (unmodified wri_op_gqa_attention from
    oracle/_ref, else the C restatement) for the 16 sessions of one GPU's share
    of the job, one session per host thread, and once on a single thread, which
    is how the reference itself runs attention.  A rate: tokens of that share
    over its time, at every --gpus N (the CPU arm has one host to run on)."""
    rank = int(os.environ.get("RANK", "0"))
    if rank != 0:
        return
    chk, kind = cpu_checker()
    threads = os.cpu_count() or 1
    lens, q, ks, vs = host_inputs(0, 1)
    for _ in range(max(args.warmup, 1)):
        cpu_decode_once(chk, q, ks, vs, threads)
    times = []
    for _ in range(args.steps):
        dt, _ = cpu_decode_once(chk, q, ks, vs, threads)
        times.append(dt)
    one_thread, _ = cpu_decode_once(chk, q, ks, vs, 1)
    total = sum(times)
    value = N_SESS * args.steps / total
    line = {
        "impl": "reference", "metric": METRIC, "value": value, "unit": UNIT,
        "n_gpus": args.gpus, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": 1e3 * total / args.steps, "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "f32 accumulate over f16 K/V", "data": "synthetic",
        "config": workload_config(args.gpus, "attention only: the reference's RoPE and KV append "
                                  "(negligible beside its attention) are not in this arm's step"),
        "cpu_baseline": {"value": value, "unit": UNIT, "cores": threads, "kind": kind,
                         "sample": "each step = attention of 16 sessions (rank 0's share at 1 GPU), one "
                                   "wri_op_gqa_attention call per session, one session per host thread; the "
                                   "op itself is scalar C (SIMD level affects matmul only)",
                         "value_1_thread": N_SESS / one_thread, "ms_per_step_1_thread": 1e3 * one_thread},
        "e2e": {"value": value, "unit": UNIT, "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
    }
    print(json.dumps(line))


def workload_config(n_gpus, note=None):
    cfg = {"workload": "c2_batched_decode", "sessions_per_gpu": N_SESS, "heads": "32Q/8KV hd128",
           "ctx": "U[1024,4096] seeded, balanced over GPUs", "step": "rope+append+decode, 1 layer",
           "parallelism": f"sessions over {n_gpus} GPU(s), no collective",
           "l2_defeat": f"rotating {N_ROT_LAYERS} layer caches, each > L2"}
    if note:
        cfg["note"] = note
    return cfg


# ------------------------------------------------- prefill (benchmark config 3)

PF_N, PF_HQ, PF_HKV = 2048, 32, 8


def measure_prefill(ctx, stream, torch, reps):
    """Causal prefill attention of one 2048-token prompt (32Q/8KV, hd 128, F16
    Q/K/V ~N(0,1)), `reps` launches back to back between two events on the
    launching stream.  flops = 4*Hq*hd*S(S+1)/2 (Q.K^T and P.V, causal half)."""
    gen = torch.Generator(device="cuda")
    gen.manual_seed(SEED + 3)
    kv = ctx.kv_create(1, PF_HKV, HD, PF_N)
    for which in (0, 1):
        rows = torch.randn((PF_N, PF_HKV, HD), generator=gen, device="cuda").to(torch.float16)
        kv.write_rows(0, which, 0, rows.view(torch.int16))
    q = torch.randn((PF_N, PF_HQ, HD), generator=gen, device="cuda").to(torch.float16)
    out = torch.empty((PF_N, PF_HQ, HD), device="cuda", dtype=torch.float32)
    for _ in range(3):
        ctx.attn_prefill(kv, 0, 0, PF_N, q, out, PF_HQ)
    ctx.sync()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record(stream)
    for _ in range(reps):
        ctx.attn_prefill(kv, 0, 0, PF_N, q, out, PF_HQ)
    b.record(stream)
    ctx.sync()
    ms = a.elapsed_time(b) / reps
    flops = 4.0 * PF_HQ * HD * PF_N * (PF_N + 1) / 2
    tflops = flops / (ms * 1e-3) / 1e12
    peak, src = 1590.0, "fallback"
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            peak, src = float(json.load(f)["bf16_tflops"]), "measured"
    finite = bool(torch.isfinite(out).all().item())
    kv.close()
    return {"workload": "c3_causal_prefill 2048 tok 32Q/8KV hd128 F16", "kernel": "attn_prefill_hd128_kernel",
            "bound": "tensor", "achieved": r4(tflops), "peak": peak, "unit": "TFLOP/s", "frac": r4(tflops / peak),
            "peak_source": f"of {src} (burst)", "frac_of_2250_spec": r4(tflops / 2250.0),
            "flops_per_launch": flops, "avg_launch_ms": r4(ms), "launches": reps,
            "traffic": NCU_TRAFFIC_PREFILL_C3, "output_finite": finite}


# ------------------------------- long-context split-KV decode (benchmark config 4)

LC_CTX = 32768


def cpu_checker_long():
    """CPU reference built with the 32768-key attention cap (the cap is a
    compile-time constant of the reference), else the restatement."""
    import oracle
    ref = oracle.reference(long_context=True)
    if ref is not None:
        return ref, "reference"
    return oracle.restatement(), "port"


def measure_split_kv(ctx, stream, torch, rank, world, reps):
    """16 sessions x 32768 cached keys (8 KV heads, hd 128, ~2.1 GB of K/V per
    layer), the KEY SEQUENCE sharded contiguously over the ranks.  One step =
    per-rank partial attention -> one NCCL all-gather of the (m, l, o) triples
    -> local merge; the fused variant replaces the all-gather and the merge by
    peer-memory stores.  Timed with events on the launching stream, max over
    ranks.  Parity: rank 0 regenerates every rank's shard of session 0 from the
    per-rank seeds and compares that session's 32 merged heads with the CPU
    reference over all 32768 keys (merge algebra src/core/kernels.c:1503-1506)."""
    from wayruntime_b200 import splitkv
    ctx.set_attn_max_seq(LC_CTX)
    lo, hi = splitkv.shard_range(LC_CTX, rank, world)
    n_local = hi - lo

    def shard_rows(gen, n):
        return torch.randn((n, HKV, HD), generator=gen, device="cuda").to(torch.float16)

    gen = torch.Generator(device="cuda")
    gen.manual_seed(SEED + 77 + rank)
    kvs = [ctx.kv_create(1, HKV, HD, max(n_local, 1)) for _ in range(N_SESS)]
    for kv in kvs:
        for which in (0, 1):
            kv.write_rows(0, which, 0, shard_rows(gen, n_local).view(torch.int16))
    q = torch.randn((N_SESS, HQ, HD), generator=gen, device="cuda", dtype=torch.float32)
    if world > 1:
        import torch.distributed as dist
        dist.broadcast(q, src=0)
    out = torch.empty_like(q)
    rows_n = N_SESS * HQ
    triples = torch.empty((rows_n, 4 + HD), dtype=torch.float32, device="cuda")
    gathered = torch.empty((world, rows_n, 4 + HD), dtype=torch.float32, device="cuda")
    batch = wr_batch(kvs)
    lens = [n_local] * N_SESS

    def step():
        splitkv.decode_split_kv(ctx, batch, 0, lens, q, out, HQ, triples=triples, gathered=gathered)

    for _ in range(3):
        step()
    ctx.sync()
    torch.cuda.synchronize()
    if world > 1:
        dist.barrier()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record(stream)
    for _ in range(reps):
        step()
    b.record(stream)
    ctx.sync()
    torch.cuda.synchronize()
    ms = a.elapsed_time(b) / reps
    if world > 1:
        t = torch.tensor([ms], device="cuda", dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        ms = float(t.item())
    finite = bool(torch.isfinite(out).all().item())

    # ---- this rank's share of the step on its own: the partial attention, no exchange (max over ranks)
    for _ in range(3):
        ctx.attn_decode_partial(batch, 0, lens, q, triples, HQ)
    ctx.sync()
    if world > 1:
        dist.barrier()
    a.record(stream)
    for _ in range(reps):
        ctx.attn_decode_partial(batch, 0, lens, q, triples, HQ)
    b.record(stream)
    ctx.sync()
    torch.cuda.synchronize()
    partial_ms = a.elapsed_time(b) / reps
    if world > 1:
        t = torch.tensor([partial_ms], device="cuda", dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        partial_ms = float(t.item())

    # ---- parity of session 0 (all heads) against the CPU reference, on rank 0
    want0 = None
    parity = None
    if rank == 0:
        ks, vs = [], []
        for r in range(world):
            g = torch.Generator(device="cuda")
            g.manual_seed(SEED + 77 + r)
            rlo, rhi = splitkv.shard_range(LC_CTX, r, world)
            ks.append(shard_rows(g, rhi - rlo).cpu().numpy().view(np.uint16))   # session 0: first two draws
            vs.append(shard_rows(g, rhi - rlo).cpu().numpy().view(np.uint16))
        chk, _kind = cpu_checker_long()
        rc, want0 = chk.decode_batch(q[:1].cpu().numpy(), [np.concatenate(ks)], [np.concatenate(vs)],
                                     threads=1, max_seq=LC_CTX)
        if rc != 0:
            raise RuntimeError(f"CPU reference attention over {LC_CTX} keys returned {rc}")
        parity = float(np.abs(out[:1].cpu().numpy() - want0).max())

    # the same step with all-gather + merge fused over NVLink peer memory; after every
    # phase the ranks agree on whether all of them succeeded, so that a failure on
    # one rank can never leave another waiting in a collective
    fused = None
    if world > 1:
        def all_ok(flag):
            t = torch.tensor([1 if flag else 0], device="cuda", dtype=torch.int32)
            dist.all_reduce(t, op=dist.ReduceOp.MIN)
            return bool(t.item())

        xchg, why = None, None
        try:
            xchg = splitkv.make_exchange(ctx, rows_n, HD)         # raises on every rank or on none
        except Exception as exc:
            why = f"{type(exc).__name__}: {exc}"
        if xchg is not None:
            out_f = torch.empty_like(q)

            def step_fused_two_kernels():
                splitkv.decode_split_kv(ctx, batch, 0, lens, q, out_f, HQ, triples=triples, exchange=xchg)

            step_fused = step_fused_two_kernels

            def run(n, end_event=None):
                try:
                    for _ in range(n):
                        step_fused()
                    if end_event is not None:
                        end_event.record(stream)
                    ctx.sync()                                     # a kernel that gave up waiting surfaces here
                    return True
                except Exception as exc:
                    nonlocal why
                    why = f"{type(exc).__name__}: {exc}"
                    return False

            good = all_ok(run(3))
            if good:
                dist.barrier()
                a.record(stream)
                good = all_ok(run(reps, b))
                torch.cuda.synchronize()
            if good:
                t = torch.tensor([a.elapsed_time(b) / reps], device="cuda", dtype=torch.float64)
                dist.all_reduce(t, op=dist.ReduceOp.MAX)
                fused = {"ms_per_step": r4(t.item()),
                         "identical_to_allgather_path": bool(torch.equal(out_f, out))}
                if want0 is not None:
                    fused["parity_max_abs_err"] = r4(np.abs(out_f[:1].cpu().numpy() - want0).max())
                # the decode kernel's own warps deliver the triples to the peers
                out_d = torch.empty_like(q)

                def step_fused_decode():
                    splitkv.decode_split_kv(ctx, batch, 0, lens, q, out_d, HQ, exchange=xchg, fused_decode=True)

                step_fused = step_fused_decode
                good = all_ok(run(3))
                if good:
                    dist.barrier()
                    a.record(stream)
                    good = all_ok(run(reps, b))
                    torch.cuda.synchronize()
                if good:
                    t = torch.tensor([a.elapsed_time(b) / reps], device="cuda", dtype=torch.float64)
                    dist.all_reduce(t, op=dist.ReduceOp.MAX)
                    fused["in_decode_kernel_ms_per_step"] = r4(t.item())
                    fused["in_decode_kernel_identical"] = bool(torch.equal(out_d, out))
                else:
                    fused["in_decode_kernel_error"] = why or "a peer rank failed"
            splitkv.close_exchange(xchg, ctx)                      # destroy is collective
        if fused is None:
            fused = {"error": why or "a peer rank failed"}
    for kv in kvs:
        kv.close()
    total_bytes = N_SESS * LC_CTX * HKV * HD * 2 * 2
    peak, src = measured_peaks()
    per_gpu = total_bytes / world / (ms * 1e-3) / 1e9
    res = {"cfg": f"c4 16x{LC_CTX} keys sharded over {world} GPU(s)", "ms_per_step": r4(ms),
           "tok_s": r4(N_SESS / (ms * 1e-3)), "hbm_gbs_per_gpu": r4(per_gpu),
           "frac_per_gpu": r4(per_gpu / peak), "peak_source": f"of {src}",
           "partial_attention_only_ms": r4(partial_ms),
           "collective": "none" if world == 1 else "NCCL all-gather of triples",
           "parity_max_abs_err": r4(parity), "parity_sample": "session 0, 32 heads, 32768 keys vs CPU reference",
           "output_finite": finite}
    if fused is not None:
        res["fused_exchange_merge"] = fused
    return res


# --------------------- KV-head-sharded serving shape (benchmark config 5)

C5_SESS, C5_PREFILL, C5_HKV, C5_GROUP = 8, 8192, 8, 5


def measure_kv_head_sharded(ctx, stream, torch, rank, world, reps):
    """8 sessions, 40Q/8KV heads, hd 128: an 8192-token causal prefill per
    session, then batched decode steps over the 8193 cached keys.  KV-head
    groups are independent (src/core/kernels.c:1477), so rank r holds
    8/world KV heads with their five Q heads each and no collective is
    needed; at one GPU it holds all eight.  Prefill: `reps` launches of one
    session's prompt; decode: 4*reps launches of the 8-session step."""
    hkv = max(1, C5_HKV // world)
    hq = hkv * C5_GROUP
    ctx.set_attn_max_seq(LC_CTX)
    gen = torch.Generator(device="cuda")
    gen.manual_seed(SEED + 55 + rank)
    n_ctx = C5_PREFILL + 1
    kvs = [ctx.kv_create(1, hkv, HD, n_ctx) for _ in range(C5_SESS)]
    for kv in kvs:
        for which in (0, 1):
            rows = torch.randn((n_ctx, hkv, HD), generator=gen, device="cuda").to(torch.float16)
            kv.write_rows(0, which, 0, rows.view(torch.int16))
    qp = torch.randn((C5_PREFILL, hq, HD), generator=gen, device="cuda").to(torch.float16)
    outp = torch.empty((C5_PREFILL, hq, HD), device="cuda", dtype=torch.float32)
    qd = torch.randn((C5_SESS, hq, HD), generator=gen, device="cuda", dtype=torch.float32)
    outd = torch.empty_like(qd)
    batch = wr_batch(kvs)
    lens = [n_ctx] * C5_SESS

    def timed(fn, n):
        for _ in range(2):
            fn(0)
        ctx.sync()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record(stream)
        for i in range(n):
            fn(i)
        b.record(stream)
        ctx.sync()
        ms = a.elapsed_time(b) / n
        if world > 1:
            import torch.distributed as dist
            t = torch.tensor([ms], device="cuda", dtype=torch.float64)
            dist.all_reduce(t, op=dist.ReduceOp.MAX)
            ms = float(t.item())
        return ms

    pf_ms = timed(lambda i: ctx.attn_prefill(kvs[i % C5_SESS], 0, 0, C5_PREFILL, qp, outp, hq), reps)
    dec_ms = timed(lambda i: ctx.attn_decode(batch, 0, lens, qd, outd, hq), 4 * reps)
    finite = bool(torch.isfinite(outp).all().item() and torch.isfinite(outd).all().item())
    # ---- parity on rank 0 (its own heads; KV-head groups are independent): session 0's
    # decode row over all 8193 keys, and a subset of session 0's prefill rows, all heads
    dec_err = pf_err = None
    if rank == 0:
        chk, _kind = cpu_checker_long()
        threads = os.cpu_count() or 1
        k0, v0 = kvs[0].read_rows(0, 0, 0, n_ctx), kvs[0].read_rows(0, 1, 0, n_ctx)
        rc, want = chk.decode_batch(qd[:1].cpu().numpy(), [k0], [v0], threads=1, max_seq=LC_CTX)
        if rc != 0:
            raise RuntimeError(f"CPU reference decode returned {rc}")
        dec_err = float(np.abs(outd[:1].cpu().numpy() - want).max())
        ctx.attn_prefill(kvs[0], 0, 0, C5_PREFILL, qp, outp, hq)
        ctx.sync()
        rows = np.array([0, 1, 63, 64, 127, 128, 1000, 4095, 4096, 8190, 8191], dtype=np.uint32)
        rc, wantp = chk.causal_prefill_rows(qp.cpu().numpy().view(np.uint16), k0[:C5_PREFILL], v0[:C5_PREFILL],
                                            rows, threads=threads, max_seq=LC_CTX)
        if rc != 0:
            raise RuntimeError(f"CPU reference prefill rows returned {rc}")
        pf_err = float(np.abs(outp.cpu().numpy()[rows] - wantp).max())
    for kv in kvs:
        kv.close()
    ctx.set_attn_max_seq(LC_CTX)
    flops = 4.0 * hq * HD * C5_PREFILL * (C5_PREFILL + 1) / 2            # per session, per rank
    dec_bytes = C5_SESS * n_ctx * hkv * HD * 2 * 2 + 2 * C5_SESS * hq * HD * 4
    peak_bw, src = measured_peaks()
    peak_tf = 1590.0
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            peak_tf = float(json.load(f)["bf16_tflops"])
    tf = flops / (pf_ms * 1e-3) / 1e12
    gbs = dec_bytes / (dec_ms * 1e-3) / 1e9
    return {"cfg": f"c5 8 sess, 8192-tok prefill + decode, {hq}Q/{hkv}KV per GPU x {world}, no collective",
            "prefill_ms_per_session": r4(pf_ms), "prefill_tflops_per_gpu": r4(tf), "prefill_frac": r4(tf / peak_tf),
            "decode_ms_per_step": r4(dec_ms), "decode_gbs_per_gpu": r4(gbs), "decode_frac": r4(gbs / peak_bw),
            "decode_tok_s": r4(C5_SESS / (dec_ms * 1e-3)), "peak_source": f"of {src}",
            "decode_parity_max_abs_err": r4(dec_err), "prefill_parity_max_abs_err": r4(pf_err),
            "parity_sample": "rank 0: session 0 decode row; 11 prefill rows; all heads",
            "output_finite": finite}


WHOLE_MODEL_SHAPE = dict(n_layers=28, hidden=1024, n_q=16, n_kv=8, head_dim=128, ffn=3072, vocab=151936)
WHOLE_MODEL_PROMPT, WHOLE_MODEL_TOKENS = 64, 32
WHOLE_MODEL_BATCH_PROMPT, WHOLE_MODEL_BATCH_STEPS = 8, 6


def measure_whole_model():
    """benchmark config 1 end to end through the public C API, `wayrt bench` style
    (src/cli/wayrt.c:694-854: prefill all prompt tokens but the last, then N
    greedy steps, wall clock around each phase), on a seeded GGUF of the
    Qwen3-0.6B shape: the unmodified reference library on the host cores, the
    drop-in library with only attention on the device (WR_B200_GLUE=host), and the
    drop-in with the whole layer stack on the device (the default)."""
    from wayruntime_b200 import wayrt_bench as wb
    ref_path = os.path.join(ROOT, "oracle", "_ref", "libwayruntime_ref.so")
    b200_path = os.path.join(ROOT, "wayruntime_b200", "lib", "libwayruntime_b200.so")
    if not (os.path.exists(ref_path) and os.path.exists(b200_path)):
        return {"unavailable": "the compiled reference and the drop-in library are built where the "
                               "reference checkout exists; neither was found beside this file"}
    sys.path.insert(0, os.path.join(ROOT, "tests"))
    import tempfile
    import _mkgguf
    shape = WHOLE_MODEL_SHAPE
    path = os.path.join(tempfile.mkdtemp(prefix="wr_bench_gguf_"), "qwen3_0p6b_shape.gguf")
    _mkgguf.write_qwen3(path, seed=SEED, **shape)
    prompt = wb.seeded_prompt(WHOLE_MODEL_PROMPT, shape["vocab"], SEED)
    out = {"workload": "c1_single_stream: Qwen3-0.6B shape (28 layers, hidden 1024, 16 Q / 8 KV heads, "
                       "head_dim 128, QK-norm, SwiGLU 3072, vocab 151936), F16 GGUF with seeded N(0, 0.02) "
                       "weights (held as F32 by the loader), "
                       f"{WHOLE_MODEL_PROMPT}-token seeded prompt, {WHOLE_MODEL_TOKENS} greedy tokens",
           "timer": "wayrt bench restated over the public C API (wayruntime_b200/wayrt_bench.py)"}
    runs = (("reference", ref_path, None), ("b200_attention_only", b200_path, "host"),
            ("b200_device_glue", b200_path, "device"))
    ids = {}
    try:
        for name, lib_path, glue in runs:
            if glue:
                os.environ["WR_B200_GLUE"] = glue
            lib = wb.Library(lib_path)
            try:
                # one short untimed pass per library first (page cache, lazy kernel loading), as for every arm
                wb.bench(lib, path, prompt[:8], 2, shape["vocab"])
                res = wb.bench(lib, path, prompt, WHOLE_MODEL_TOKENS, shape["vocab"])
            finally:
                lib.close()
            ids[name] = res["ids"]
            out[name] = {"prefill_tok_s": r4(wb.rate(res["n_prefill"], res["prefill_s"])),
                         "prefill_ms": r4(1e3 * res["prefill_s"]),
                         "decode_tok_s": r4(wb.rate(res["produced"], res["decode_s"])),
                         "decode_ms_per_token": r4(1e3 * res["decode_s"] / max(1, res["produced"])),
                         "threads": res["threads"],
                         "attention_calls": res["counters"][3], "matmul_calls": res["counters"][0]}
    finally:
        os.environ.pop("WR_B200_GLUE", None)
        batch_path = path + ".batch"
        os.replace(path, batch_path)                      # kept for the batched section below
    # the batched step (wr_batch_step, 16 sessions): reference against the device layer stack
    try:
        bprompts = [wb.seeded_prompt(WHOLE_MODEL_BATCH_PROMPT + i, shape["vocab"], SEED + 100 + i)
                    for i in range(N_SESS)]
        batch = {}
        for name, lib_path, glue in (("reference", ref_path, None), ("b200_device_glue", b200_path, "device")):
            if glue:
                os.environ["WR_B200_GLUE"] = glue
            lib = wb.Library(lib_path)
            try:
                rb = wb.bench_batch(lib, batch_path, bprompts, WHOLE_MODEL_BATCH_STEPS, shape["vocab"])
            finally:
                lib.close()
                os.environ.pop("WR_B200_GLUE", None)
            batch[name] = {"decode_tok_s": r4(wb.rate(rb["sessions"] * rb["steps"], rb["decode_s"])),
                           "ms_per_batched_step": r4(1e3 * rb["decode_s"] / rb["steps"]),
                           "prefill_tok_s": r4(wb.rate(rb["n_prefill"], rb["prefill_s"])), "ids": rb["ids"]}
        same_b = sum(a == b for a, b in zip(batch["reference"].pop("ids"), batch["b200_device_glue"].pop("ids")))
        batch["workload"] = (f"wr_batch_step, {N_SESS} sessions, prompts of {WHOLE_MODEL_BATCH_PROMPT}-"
                             f"{WHOLE_MODEL_BATCH_PROMPT + N_SESS - 1} tokens, {WHOLE_MODEL_BATCH_STEPS} greedy steps")
        batch["sessions_with_identical_greedy_ids"] = f"{same_b} of {N_SESS}"
        batch["decode_speedup_vs_reference"] = r4(batch["b200_device_glue"]["decode_tok_s"] /
                                                  batch["reference"]["decode_tok_s"])
        out["batched_step"] = batch
    except Exception as exc:
        out["batched_step"] = {"error": f"{type(exc).__name__}: {exc}"}
    finally:
        if os.path.exists(batch_path):
            os.remove(batch_path)
    for name in ("b200_attention_only", "b200_device_glue"):
        same = 0
        for a, b in zip(ids["reference"], ids[name]):
            if a != b:
                break
            same += 1
        out[name]["greedy_ids_equal_to_reference"] = f"{same} of {len(ids['reference'])} (free-running)"
        out[name]["decode_speedup_vs_reference"] = r4(out[name]["decode_tok_s"] / out["reference"]["decode_tok_s"])
        out[name]["prefill_speedup_vs_reference"] = r4(out[name]["prefill_tok_s"] / out["reference"]["prefill_tok_s"])
    return out


# ---- models whose layers differ (Tumadra, Nurosun), beside the dense stack at the same width, depth and widths of the parts

MIXED_SIZES = {
    # name: width, layers, ff, query heads, kv heads, inner, dt_rank, vocab
    "w1024x28": (1024, 28, 3072, 8, 4, 2048, 64, 151936),
    "w2048x12": (2048, 12, 6144, 16, 4, 4096, 128, 65536),
    "w4096x4": (4096, 4, 12288, 32, 8, 8192, 256, 65536),
}
MIXED_PREFILL, MIXED_CTX = 2048, 1024


class PooledWeights:
    """Random weights of any shape cut from one small pool (the timing does not depend on the values)."""

    def __init__(self, bf16):
        from wayruntime_b200.checkpoint import f32_to_bf16
        pool = np.random.default_rng(SEED).standard_normal((1 << 22) + 7).astype(np.float32) * 0.02
        self.pool, self.bf16 = (f32_to_bf16(pool) if bf16 else pool), bf16

    def get(self, name, shape):
        if "norm" in name or name.endswith((".D", "shift")):
            a = np.full(shape, 1.0 if "norm" in name else 0.5, np.float32)
            from wayruntime_b200.checkpoint import f32_to_bf16
            return f32_to_bf16(a) if self.bf16 else a
        return np.resize(self.pool, shape)

    f32 = get

    def __contains__(self, name):
        return True


def mixed_config(size):
    width, n, ff, heads, kv, inner, rank, vocab = MIXED_SIZES[size]
    attn = {"type": "attention", "mlp": {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv, "dim": 64, "vdim": 128, "scale": 0.125, "diff": 0.5,
                      "q_temp": {"coef": 0.1, "every": 1024}}}
    scan = {"type": "mamba1", "mlp": {"kind": "dense", "ff": ff},
            "mixer": {"inner": inner, "state": 16, "dt_rank": rank, "conv": 4}}
    return {"architecture": "Tumadra", "width": width, "vocab": vocab, "norm": {"groups": 4, "eps": 1e-5},
            "layers": [attn if i % 2 else scan for i in range(n)]}


def latent_config(size):
    """Nurosun: pairs of a layer with rows of its own and a dense feed-forward, and one that borrows them and has
    experts, of which a token uses as much as the dense layer is wide."""
    width, n, ff, heads, _kv, _inner, _rank, vocab = MIXED_SIZES[size]
    mixer = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": width // 2, "kv_rank": 512, "scale": 192 ** -0.5,
             "rot": {"base": 10000.0, "dims": 64}}
    moe = {"kind": "moe", "expert": {"ff": ff // 4, "limit": 7.0}, "router": {"experts": 32, "top": 4}}
    layers = [{"type": "latent_attention", "mixer": dict(mixer, kv_from=i - 1), "mlp": moe} if i % 2 else
              {"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff}} for i in range(n)]
    return {"architecture": "Nurosun", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "embedding": {"scale": width ** 0.5},
            "residual_mult": 0.5, "layers": layers}


def dense_config(size):
    width, n, ff, heads, kv, _inner, _rank, vocab = MIXED_SIZES[size]
    return {"architectures": ["Qwen3ForCausalLM"], "hidden_size": width, "intermediate_size": ff, "num_hidden_layers": n,
            "num_attention_heads": heads, "num_key_value_heads": kv, "head_dim": 128, "vocab_size": vocab,
            "tie_word_embeddings": True, "rope_theta": 1e6, "rms_norm_eps": 1e-6}


def measure_mixed(args):
    """Prefill and decode throughput of mixed models (BF16) and of the dense F32 stack at equal size, each through
    its forward call: prefill of MIXED_PREFILL tokens, decode of 1 and 16 sessions at MIXED_CTX tokens, arg-max on the
    device, CUDA events on the context's stream around the calls (host enqueueing included)."""
    import torch
    import wayruntime_b200 as wr
    from wayruntime_b200 import models
    out = {"only": "mixed", "prefill_tokens": MIXED_PREFILL, "decode_context": MIXED_CTX, "data": "synthetic",
           "weights": "random, repeated from one pool", "sizes": {}}
    rng = np.random.default_rng(SEED)
    for size in (args.mixed_size.split(",") if args.mixed_size else MIXED_SIZES):
        row = out["sizes"][size] = {}
        for kind, cfg, dtype, rows in (("nurosun_bf16", latent_config(size), "bfloat16", MIXED_PREFILL),
                                       ("tumadra_bf16", mixed_config(size), "bfloat16", MIXED_PREFILL),
                                       ("dense_f32", dense_config(size), "float32", 256)):
            if args.mixed_kind and kind != args.mixed_kind:
                continue
            ctx = wr.Context(0)
            stream = torch.cuda.ExternalStream(ctx.stream, device=0)
            m = models.build(ctx, cfg, PooledWeights(dtype == "bfloat16"), dtype, rows)
            vocab = m.vocab
            toks = [int(t) for t in rng.integers(0, vocab, MIXED_PREFILL)]

            def timed(fn, reps):
                ev = [torch.cuda.Event(enable_timing=True) for _ in range(2)]
                ms = []
                for _ in range(reps):
                    ev[0].record(stream)
                    fn()
                    ev[1].record(stream)
                    ev[1].synchronize()
                    ms.append(ev[0].elapsed_time(ev[1]))
                return float(np.median(ms))

            kv = m.kv_create(MIXED_PREFILL + 8)

            def prefill():
                for lo in range(0, MIXED_PREFILL, rows):
                    part = toks[lo:lo + rows]
                    last = lo + len(part) == MIXED_PREFILL
                    m.forward(m.FWD_PREFILL, [kv], [lo], part, out_from=len(part) - 1, argmax=last)
            reps = max(3, min(args.steps, 20))
            timed(prefill, 2)
            ms = timed(prefill, reps)
            kv.close()
            res = row[kind] = {"device_weight_bytes": m.device_bytes, "prefill_ms": r4(ms),
                               "prefill_tok_s": r4(MIXED_PREFILL / ms * 1e3)}
            for n in (1, 16):
                kvs = [m.kv_create(MIXED_CTX + 256) for _ in range(n)]
                for kv in kvs:
                    for lo in range(0, MIXED_CTX, rows):
                        part = toks[lo:min(lo + rows, MIXED_CTX)]
                        m.forward(m.FWD_PREFILL, [kv], [lo], part, out_from=len(part))
                pos = [MIXED_CTX]

                def decode():
                    m.forward(m.FWD_DECODE, kvs, [pos[0]] * n, toks[:n], argmax=True)
                    pos[0] += 1
                timed(decode, 5)
                l0 = m.launches
                ms = timed(decode, args.mixed_reps)
                res[f"decode_{n}"] = {"ms": r4(ms), "tok_s": r4(n / ms * 1e3), "enqueue_ms": r4(m.last_enqueue_ms),
                                      "launches": (m.launches - l0) // args.mixed_reps}
                for kv in kvs:
                    kv.close()
            m.close()
            ctx.close()
    print(json.dumps(out))


def wr_batch(kvs):
    import wayruntime_b200 as wr
    return wr.Batch(kvs)


# ----------------------------------------------------------------- GPU arm

def run_gpu_arm(args):
    import torch
    import wayruntime_b200 as wr

    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    json_out = sys.stdout
    if world > 1:
        import torch.distributed as dist
        # stdout carries exactly one JSON line: whatever NCCL (a C library) writes to file
        # descriptor 1 goes to stderr instead; the line itself is written to the saved descriptor
        sys.stdout.flush()
        json_out = os.fdopen(os.dup(1), "w")
        os.dup2(2, 1)
        torch.cuda.set_device(local)
        dist.init_process_group("nccl", device_id=torch.device("cuda", local))
    torch.cuda.set_device(local)
    if wr.device_check(local) != 0:
        raise SystemExit("no sm_100 device bound: wayruntime_b200 has no CPU path")

    ctx = wr.Context(local)
    stream = torch.cuda.ExternalStream(ctx.stream, device=local)
    if args.only == "prefill":
        # profiling aid: just the prefill kernel, a few launches, one short JSON line
        torch.cuda.set_stream(stream)
        res = measure_prefill(ctx, stream, torch, max(1, args.steps))
        if rank == 0:
            print(json.dumps({"only": "prefill", "roofline_prefill": res}))
        ctx.close()
        return
    lens = session_lengths(rank, world)
    positions = [n - 1 for n in lens]

    # ---- device-resident synthetic caches
    gen = torch.Generator(device="cuda")
    gen.manual_seed(SEED + rank)
    kvs = [ctx.kv_create(N_ROT_LAYERS, HKV, HD, CTX_HI) for _ in lens]
    for kv, n in zip(kvs, lens):
        for layer in range(N_ROT_LAYERS):
            for which in (0, 1):
                rows = torch.randn((n, HKV, HD), generator=gen, device="cuda",
                                   dtype=torch.float32).to(torch.float16)
                kv.write_rows(layer, which, 0, rows.view(torch.int16))
    ctx.sync()
    q_src = torch.randn((N_SESS, HQ, HD), generator=gen, device="cuda", dtype=torch.float32)
    k_new = torch.randn((N_SESS, HKV, HD), generator=gen, device="cuda", dtype=torch.float32)
    v_new = torch.randn((N_SESS, HKV, HD), generator=gen, device="cuda", dtype=torch.float32)
    q_work = torch.empty_like(q_src)
    out = torch.empty_like(q_src)
    torch.cuda.synchronize()

    batch = wr.Batch(kvs)
    pos_arr = wr.Batch.u32(positions)
    len_arr = wr.Batch.u32(lens)

    torch.cuda.set_stream(stream)       # torch copies below go on the context's stream

    if args.only == "decode":
        # profiling aid: just the decode kernel on the config-2 batch, launched eagerly
        for i in range(max(args.warmup, 1)):
            ctx.attn_decode(batch, i % N_ROT_LAYERS, len_arr, q_src, out, HQ)
        ctx.sync()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record(stream)
        for i in range(args.steps):
            ctx.attn_decode(batch, i % N_ROT_LAYERS, len_arr, q_src, out, HQ)
        b.record(stream)
        ctx.sync()
        ms = a.elapsed_time(b) / args.steps
        alg = algorithmic_bytes(lens)
        if rank == 0:
            print(json.dumps({"only": "decode", "avg_launch_ms": r4(ms), "algorithmic_bytes_per_launch": alg,
                              "achieved_gbs": r4(alg / (ms * 1e-3) / 1e9), "launch_mode": "eager"}))
        for kv in kvs:
            kv.close()
        ctx.close()
        return

    def step_device(i):
        # A fresh un-rotated Q each step (device-to-device, 256 KB), then RoPE +
        # append + decode of one layer in one C-ABI call.
        q_work.copy_(q_src, non_blocking=True)
        ctx.decode_step(batch, i % N_ROT_LAYERS, pos_arr, q_work, k_new, v_new, out, HQ,
                        theta=THETA)

    def barrier():
        if world > 1:
            import torch.distributed as dist
            dist.barrier()
        torch.cuda.synchronize()

    def max_over_ranks(x):
        if world == 1:
            return x
        import torch.distributed as dist
        t = torch.tensor([x], device="cuda", dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        return float(t.item())

    # cached keys streamed per step by the whole job
    if world > 1:
        import torch.distributed as dist
        tsum = torch.tensor([float(sum(lens))], device="cuda", dtype=torch.float64)
        dist.all_reduce(tsum, op=dist.ReduceOp.SUM)
        job_sum_ctx = float(tsum.item())
    else:
        job_sum_ctx = float(sum(lens))

    # ---- warm-up, then the device-resident timed region
    for i in range(args.warmup):
        step_device(i)
    ctx.sync()
    # The step is launch-bound from Python (tens of microseconds of work per
    # step), so one pass over the rotating layers is captured in a CUDA graph
    # and replayed; leftover steps run eagerly.
    graph, launch_mode = None, "eager"
    l_cap = ctx.launch_count
    if not args.no_graph:
        try:
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph, stream=stream, capture_error_mode="thread_local"):
                for i in range(N_ROT_LAYERS):
                    step_device(i)
            launch_mode = f"cuda graph of {N_ROT_LAYERS} steps"
        except Exception as exc:          # capture unavailable: measure eagerly, say so
            graph, launch_mode = None, f"eager (graph capture failed: {type(exc).__name__})"
            torch.cuda.synchronize()
    launches_per_step = (ctx.launch_count - l_cap) / N_ROT_LAYERS if graph else None
    torch.cuda.set_stream(stream)
    if graph is not None:
        graph.replay()
    ctx.sync()
    sampler = ClockSampler(local)
    if rank == 0:
        sampler.start()

    def k_steps():
        n_replay = args.steps // N_ROT_LAYERS if graph is not None else 0
        for _ in range(n_replay):
            graph.replay()
        for i in range(n_replay * N_ROT_LAYERS, args.steps):
            step_device(i)
        return n_replay

    # One probe repetition sizes the region; then the K-step region is repeated back to
    # back, an event between repetitions, until at least MIN_TIMED_S of device time is
    # covered.  The figure reported is the median repetition (max over ranks per repetition).
    pa, pb = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    pa.record(stream)
    k_steps()
    pb.record(stream)
    ctx.sync()
    probe_ms = max(pa.elapsed_time(pb), 1e-3)
    n_reps = int(max(1, min(2000, np.ceil(MIN_TIMED_S * 1e3 / probe_ms))))
    if world > 1:
        import torch.distributed as dist
        t = torch.tensor([n_reps], device="cuda", dtype=torch.int64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        n_reps = int(t.item())
    barrier()
    l0 = ctx.launch_count
    marks = [torch.cuda.Event(enable_timing=True) for _ in range(n_reps + 1)]
    marks[0].record(stream)
    n_replay = 0
    for r in range(n_reps):
        n_replay = k_steps()
        marks[r + 1].record(stream)
    ctx.sync()
    barrier()
    launches = ctx.launch_count - l0                    # whole timed region: n_reps x K steps
    if graph is not None:
        launches += int(launches_per_step * n_replay * N_ROT_LAYERS) * n_reps
    rep_ms = torch.tensor([marks[r].elapsed_time(marks[r + 1]) for r in range(n_reps)],
                          device="cuda", dtype=torch.float64)
    if world > 1:
        dist.all_reduce(rep_ms, op=dist.ReduceOp.MAX)
    timed_region_s = float(rep_ms.sum().item()) * 1e-3
    step_ms = float(rep_ms.median().item()) / args.steps
    step_ms_spread = [float(rep_ms.min().item()) / args.steps, float(rep_ms.max().item()) / args.steps]

    # ---- decode kernel alone (roofline): K launches back to back between two
    # events on the launching stream, rotating layers; average per launch
    def decode_only(i):
        ctx.attn_decode(batch, i % N_ROT_LAYERS, len_arr, q_work, out, HQ)

    dgraph = None
    if graph is not None:
        try:
            dgraph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(dgraph, stream=stream, capture_error_mode="thread_local"):
                for i in range(N_ROT_LAYERS):
                    decode_only(i)
        except Exception:
            dgraph = None
            torch.cuda.synchronize()
    torch.cuda.set_stream(stream)
    for i in range(N_ROT_LAYERS):
        decode_only(i)
    ctx.sync()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record(stream)
    n_rep = args.steps // N_ROT_LAYERS if dgraph is not None else 0
    dec_reps = max(1, n_reps // 2)
    for _ in range(dec_reps):
        for _ in range(n_rep):
            dgraph.replay()
        for i in range(n_rep * N_ROT_LAYERS, args.steps):
            decode_only(i)
    b.record(stream)
    ctx.sync()
    dec_avg_ms = a.elapsed_time(b) / (args.steps * dec_reps)
    # nvidia-smi reports every 50 ms and a short run (K steps of ~40 us) ends before its
    # second report: the same step loop is kept running, untimed, until half a second of
    # this load has been sampled, so that the clock record describes the timed kernels.
    t_soak = time.perf_counter()
    while time.perf_counter() - t_soak < 0.5:
        for _ in range(64):
            if graph is not None:
                graph.replay()
            else:
                step_device(0)
        ctx.sync()
    clocks = sampler.stop() if rank == 0 else None
    if clocks is not None:
        clocks["window"] = "timed steps + 0.5 s of the same step loop"

    # ---- end to end through the C-ABI with pinned host buffers
    hq_src = torch.randn((N_SESS, HQ, HD), dtype=torch.float32).pin_memory()
    hk = torch.randn((N_SESS, HKV, HD), dtype=torch.float32).pin_memory()
    hv = torch.randn((N_SESS, HKV, HD), dtype=torch.float32).pin_memory()
    hout = torch.empty((N_SESS, HQ, HD), dtype=torch.float32).pin_memory()

    # the call a C host makes: arguments are pointers it already holds, so they are resolved once
    host_step = ctx.prepared_decode_step(batch, pos_arr, hq_src, hk, hv, hout, HQ, theta=THETA)
    hout_view = hout.numpy()

    def step_host(i):
        # Host Q/K/V in, attention rows out: copies and sync are inside the call.
        host_step(i % N_ROT_LAYERS)
        return float(hout_view[0, 0, 0])                # the step's result is read on the host

    for i in range(max(args.warmup, 3)):
        step_host(i)
    barrier()
    e2e_steps = args.steps * n_reps                     # as much work as the device-resident region
    t0 = time.perf_counter()
    for i in range(e2e_steps):
        step_host(i)
    ctx.sync()
    e2e_s = max_over_ranks(time.perf_counter() - t0)
    kv_row_bytes = N_SESS * HKV * HD * 4
    q_bytes = N_SESS * HQ * HD * 4
    h2d = 2 * kv_row_bytes + q_bytes
    d2h = q_bytes

    prefill = measure_prefill(ctx, stream, torch, max(10, min(args.steps, 50))) if rank == 0 else None
    try:
        split_kv = measure_split_kv(ctx, stream, torch, rank, world, 10)
    except Exception as exc:                       # reported, never fatal for the headline line
        split_kv = {"error": f"{type(exc).__name__}: {exc}"}
        if world > 1:
            raise

    try:
        kv_head_sharded = measure_kv_head_sharded(ctx, stream, torch, rank, world, 5)
    except Exception as exc:
        kv_head_sharded = {"error": f"{type(exc).__name__}: {exc}"}
        if world > 1:
            raise

    whole_model = None
    if rank == 0 and world == 1 and not args.no_whole_model:
        try:
            whole_model = measure_whole_model()
        except Exception as exc:
            whole_model = {"error": f"{type(exc).__name__}: {exc}"}

    # ---- parity spot check + CPU baseline on rank 0 (bounded sample)
    cpu = None
    max_err = None
    if rank == 0:
        chk, kind = cpu_checker()
        threads = os.cpu_count() or 1
        layer = 0
        sample = list(range(N_SESS)) if world == 1 else [0, 1]     # N > 1: two sessions, parity only
        ks = [kvs[i].read_rows(layer, 0, 0, lens[i]) for i in sample]
        vs = [kvs[i].read_rows(layer, 1, 0, lens[i]) for i in sample]
        ctx.attn_decode(kvs, layer, lens, q_work, out, HQ)
        ctx.sync()
        q_host = q_work.cpu().numpy()[sample]
        got = out.cpu().numpy()[sample]
        cpu_decode_once(chk, q_host, ks, vs, threads)                      # warm-up
        reps = [cpu_decode_once(chk, q_host, ks, vs, threads) for _ in range(3 if world == 1 else 1)]
        max_err = float(np.abs(reps[0][1] - got).max())
        if world == 1:
            best = min(r[0] for r in reps)
            one_thread, _ = cpu_decode_once(chk, q_host, ks, vs, 1)
            cpu = {"value": r4(N_SESS / best), "unit": UNIT, "cores": threads, "kind": kind,
                   "sample": "attention of the whole 16-session step, one session per host thread, best "
                             "of 3; once more on 1 thread (how the reference runs attention); the op is "
                             "scalar C, SIMD level affects matmul only",
                   "ms_per_step": r4(1e3 * best), "value_1_thread": r4(N_SESS / one_thread),
                   "ms_per_step_1_thread": r4(1e3 * one_thread)}

    if rank == 0:
        peak, peak_src = measured_peaks()
        alg = algorithmic_bytes(lens)
        achieved = alg / (dec_avg_ms * 1e-3) / 1e9
        sum_ctx_job = int(job_sum_ctx)
        line = {
            "metric": METRIC, "value": N_SESS * world / (step_ms * 1e-3), "unit": UNIT,
            "n_gpus": world, "steps": args.steps, "warmup": args.warmup, "ms_per_step": step_ms,
            "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
            "dtype": "f16 K/V, f32 accumulate", "data": "synthetic",
            "config": workload_config(world),
            "e2e": {"value": N_SESS * world * e2e_steps / e2e_s, "unit": UNIT,
                    "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": d2h,
                    "ms_per_step": r4(1e3 * e2e_s / e2e_steps), "steps_timed": e2e_steps},
            "gpu_launches": int(launches), "launch_mode": launch_mode,
            "repetitions": n_reps, "timed_region_s": r4(timed_region_s),
            "ms_per_step_min_max": [r4(x) for x in step_ms_spread],
            "aggregate_kv_gbs": r4(sum_ctx_job * HKV * HD * 4 / (step_ms * 1e-3) / 1e9),
            "sum_ctx": int(sum(lens)), "sum_ctx_job": sum_ctx_job,
            "clocks": clocks,
            "roofline": {"bound": "hbm", "kernel": "attn_decode_hd128_kernel",
                         "achieved": r4(achieved), "peak": peak, "unit": "GB/s",
                         "frac": r4(achieved / peak), "peak_source": f"of {peak_src}",
                         "algorithmic_bytes_per_launch": alg, "avg_launch_ms": r4(dec_avg_ms),
                         "traffic": NCU_TRAFFIC_DECODE_C2,
                         "traffic_source": "profiles/ (ncu dram read+write per launch, this workload)",
                         "frac_of_8TBs_spec": r4(achieved / 8000.0)},
            "cpu_baseline": cpu,
            "parity_max_abs_err": r4(max_err),
            "roofline_prefill": prefill,
            "whole_model": whole_model,
            # the two multi-GPU sections go last: a reader of the line's tail sees them
            "kv_head_sharded": kv_head_sharded,
            "split_kv": split_kv,
        }
        json_out.write(json.dumps(line) + "\n")
        json_out.flush()
    for kv in kvs:
        kv.close()
    ctx.close()
    if world > 1:
        import torch.distributed as dist
        dist.destroy_process_group()


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=200)
    ap.add_argument("--warmup", type=int, default=10)
    ap.add_argument("--impl", default="b200", choices=["b200", "reference"])
    ap.add_argument("--no-graph", action="store_true",
                    help="launch every step from Python instead of replaying a CUDA graph")
    ap.add_argument("--no-whole-model", action="store_true",
                    help="skip the config-1 whole-model section (about a minute of host time)")
    ap.add_argument("--only", default="all", choices=["all", "prefill", "decode", "mixed"],
                    help="'prefill' / 'decode': run only that kernel's measurement (for profiling); 'mixed': Nurosun and Tumadra "
                         "models beside the dense stack at equal size, nothing else")
    ap.add_argument("--mixed-size", default="", help="with --only mixed: sizes, with commas between them")
    ap.add_argument("--mixed-reps", type=int, default=50, help="with --only mixed: timed decode steps")
    ap.add_argument("--mixed-kind", default="", choices=["", "nurosun_bf16", "tumadra_bf16", "dense_f32"], help="with --only mixed: one model only")
    args = ap.parse_args()
    if args.impl == "reference":
        if args.steps > 20:
            args.steps = 20            # bounded sample: each step is a full 16-session pass
        run_reference_arm(args)
    elif args.only == "mixed":
        measure_mixed(args)
    else:
        run_gpu_arm(args)


if __name__ == "__main__":
    main()
