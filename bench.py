#!/usr/bin/env python
"""Headline benchmark: Q8_0 GEMV (decode) bandwidth on B200, plus the Phi-3-mini decode step.

    python bench.py [--gpus N] [--steps K] [--warmup W] [--impl ours|reference]

A "step" is one pass of the hot path over one batch of synthetic input: one GEMV
y[N] = W[N,K] . x[K] with W in ratchet's Q8_0 segment layout (f32 block scales, f16 activations),
K=16384, N=65536 — the largest shape of the GEMV sweep, 1.2 GB of weights, far larger than L2 so no
flush is needed between timed steps.  With N GPUs the rows of W are split evenly (ratchet's
"column" shard of x.W), every rank runs the GEMV on its shard and the f16 outputs are all-gathered.

Prints ONE JSON line (rank 0).  `value` is algorithmic GB/s of the whole job with inputs resident in
HBM; `e2e` is the same metric through the package's public call with the activation copied from
pinned host memory and the result copied back every step.
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
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

K_HEAD, N_HEAD = 16384, 65536
WORKLOAD = "q8_0_gemv_K16384_N65536_f16act_f32scale"


def gemv_bytes(N, K, scale_bytes=4, act_bytes=2):
    """Algorithmic bytes of one Q8_0 GEMV: int8 weights + block scales + activation + output."""
    return N * K + (N * K // 32) * scale_bytes + K * act_bytes + N * act_bytes


def measured_peak():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        with open(p) as f:
            return float(json.load(f)["hbm_gbs"]), "measured"
    return 6650.0, "fallback"


class ClockSampler:
    """Samples SM clock and clock-event (throttle) reasons through NVML every few milliseconds on a
    background thread while the timed region runs (read-only queries; nothing is set)."""

    def __init__(self, index: int, period_s: float = 0.002):
        self.index = index
        self.period = period_s
        self.samples = []   # (sm_mhz, reasons_bitmask)
        self.max_mhz = None
        self._stop = threading.Event()
        self.thread = None
        self.nvml = None

    def start(self):
        try:
            import pynvml
            pynvml.nvmlInit()
            self.nvml = pynvml
            # honour CUDA_VISIBLE_DEVICES: map the CUDA ordinal to the NVML device by UUID
            import torch
            uuid = str(torch.cuda.get_device_properties(self.index).uuid)
            try:
                self.handle = pynvml.nvmlDeviceGetHandleByUUID(("GPU-" + uuid).encode())
            except Exception:
                self.handle = pynvml.nvmlDeviceGetHandleByIndex(self.index)
            self.max_mhz = float(pynvml.nvmlDeviceGetMaxClockInfo(self.handle, pynvml.NVML_CLOCK_SM))
        except Exception:
            self.nvml = None
            return
        self.thread = threading.Thread(target=self._run, daemon=True)
        self.thread.start()

    def _run(self):
        nv = self.nvml
        while not self._stop.is_set():
            try:
                mhz = nv.nvmlDeviceGetClockInfo(self.handle, nv.NVML_CLOCK_SM)
                reasons = nv.nvmlDeviceGetCurrentClocksEventReasons(self.handle)
                self.samples.append((float(mhz), int(reasons)))
            except Exception:
                pass
            time.sleep(self.period)

    def mark(self):
        """Index of the next sample: brackets the timed region inside the sample list."""
        return len(self.samples)

    def stop(self, lo=0, hi=None):
        if self.nvml is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        self._stop.set()
        self.thread.join(timeout=2)
        nv = self.nvml
        window = self.samples[lo:hi] or self.samples
        names = {"hw_slowdown": nv.nvmlClocksEventReasonHwSlowdown, "hw_thermal_slowdown": nv.nvmlClocksEventReasonHwThermalSlowdown,
                 "sw_thermal_slowdown": nv.nvmlClocksEventReasonSwThermalSlowdown, "sw_power_cap": nv.nvmlClocksEventReasonSwPowerCap}
        reasons = [n for n, bit in names.items() if any(r & bit for _, r in window)]
        sm = [m for m, _ in window]
        return {"sm_mhz": float(np.median(sm)) if sm else None, "sm_max_mhz": self.max_mhz, "reasons": reasons,
                "samples": len(window)}


UNIQUE_ROWS = 4096


def unique_rows(K, seed):
    """The 4096 distinct rows W ~ N(0, 0.02) every benchmark matrix is made of (the values do not affect the
    timing; repeating them keeps host-side generation of a 1 Gi-element matrix to seconds and lets the
    oracle check every output row against 4096 reference values)."""
    rng = np.random.Generator(np.random.PCG64(seed))
    return rng.standard_normal((UNIQUE_ROWS, K), dtype=np.float32) * np.float32(0.02)


def make_weights(N, K, seed):
    """Synthetic Q8_0F weight buffer for W[N,K]: `unique_rows(K, seed)` quantised by the library's own
    quantiser (rcu_quantize, ratchet-core/src/quant.rs:19-99) and repeated down the matrix."""
    from ratchet_b200 import capi
    uniq = min(N, UNIQUE_ROWS)
    small = capi.quantize(unique_rows(K, seed)[:uniq])
    if uniq == N:
        return small
    off_small = capi.dtype_segments(capi.Q8_0F, uniq * K)[1]
    off = capi.dtype_segments(capi.Q8_0F, N * K)[1]
    buf = np.zeros(capi.dtype_nbytes(capi.Q8_0F, N * K), np.uint8)
    reps, rest = divmod(N, uniq)
    buf[: reps * uniq * K].reshape(reps, uniq * K)[:] = small[: uniq * K]
    buf[off: off + reps * uniq * K // 8].reshape(reps, uniq * K // 8)[:] = small[off_small: off_small + uniq * K // 8]
    if rest:
        buf[reps * uniq * K: N * K] = small[: rest * K]
        buf[off + reps * uniq * K // 8: off + N * K // 8] = small[off_small: off_small + rest * K // 8]
    return buf


def parity_report(got, ref, rtol, atol):
    """Max absolute / relative error and the count outside the reference's all_close criterion
    |a - b| <= atol + rtol * |b| (ratchet-core/src/tensor.rs:1039-1043)."""
    got = np.asarray(got, np.float64).reshape(-1)
    ref = np.asarray(ref, np.float64).reshape(-1)
    err = np.abs(got - ref)
    scale = float(np.sqrt(np.mean(ref * ref)))
    return {"max_abs": float(err.max()), "max_rel_to_rms": float(err.max() / (scale + 1e-30)),
            "outside_allclose": int((err > atol + rtol * np.abs(ref)).sum()), "rtol": rtol, "atol": atol, "checked": int(ref.size)}


def run_reference(args):
    """Reference arm: the reference's CPU path for this op (dequantise + matmul, restated in
    oracle/), all host threads, on a bounded row sample of the same workload."""
    rank = int(os.environ.get("RANK", "0"))
    if rank != 0:
        return
    from oracle import oracle as orc
    # all host cores, whatever the launcher exported (torchrun sets OMP_NUM_THREADS=1 for its workers)
    orc.set_num_threads(os.cpu_count() or 1)
    K, N = K_HEAD, N_HEAD
    rows = 2048   # 32 MiB of int8 weights per step: a bounded sample of the 65536 rows
    buf_full_rows = rows
    rng = np.random.Generator(np.random.PCG64(0))
    w = (rng.standard_normal((buf_full_rows, K), dtype=np.float32) * np.float32(0.02))
    wq = orc.quantize_q8(w)
    x = rng.standard_normal(K).astype(np.float16)
    for _ in range(args.warmup):
        orc.gemv_q8(wq, rows, K, False, x)
    t0 = time.perf_counter()
    for _ in range(args.steps):
        orc.gemv_q8(wq, rows, K, False, x)
    dt = (time.perf_counter() - t0) / args.steps
    gbs = gemv_bytes(rows, K) / dt / 1e9
    line = {
        "impl": "reference", "metric": "q8_0_gemv_gbs", "value": gbs, "unit": "GB/s", "n_gpus": args.gpus, "steps": args.steps,
        "warmup": args.warmup, "ms_per_step": dt * 1e3 * (N / rows), "higher_is_better": True, "scaling": "strong",
        "vs_baseline": None, "dtype": "i8xf16->f32", "data": "synthetic",
        "config": {"workload": WORKLOAD, "K": K, "N": N, "note": "CPU arm times a 2048-row sample; ms_per_step is scaled to all rows"},
        "cpu_baseline": {"value": gbs, "unit": "GB/s", "cores": orc.num_threads(), "kind": "port",
                         "sample": f"{rows} of {N} rows per step, {args.steps} steps"},
        "e2e": {"value": gbs, "unit": "GB/s", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
    }
    print(json.dumps(line))


def cpu_baseline_sample(K, N):
    from oracle import oracle as orc
    orc.set_num_threads(os.cpu_count() or 1)
    rows = 2048
    rng = np.random.Generator(np.random.PCG64(1))
    wq = orc.quantize_q8(rng.standard_normal((rows, K), dtype=np.float32) * np.float32(0.02))
    x = rng.standard_normal(K).astype(np.float16)
    orc.gemv_q8(wq, rows, K, False, x)
    reps, t0 = 0, time.perf_counter()
    while time.perf_counter() - t0 < 10.0 and reps < 200:
        orc.gemv_q8(wq, rows, K, False, x)
        reps += 1
    dt = (time.perf_counter() - t0) / reps
    return {"value": gemv_bytes(rows, K) / dt / 1e9, "unit": "GB/s", "cores": orc.num_threads(), "kind": "port",
            "sample": f"{rows} of {N} rows, {reps} repetitions (~10 s)"}


# DRAM bytes per weight row of the headline GEMV (K=16384): (dram__bytes_read.sum + dram__bytes_write.sum) / rows
# of an ncu capture of the same kernel on an 8192-row matrix (134 MB, larger than L2; traffic grows with rows).
GEMV_TRAFFIC_PER_ROW_BYTES = (151.075e6 + 4.9e6) / 8192

SWEEP_SHAPES = [(3072, 3072), (3072, 16384), (8192, 3072)]   # (K, N) of the decode sweep below the headline shape


def _time_loop(torch, stream, fn, iters):
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    stream.synchronize()
    e0.record(stream)
    for i in range(iters):
        fn(i)
    e1.record(stream)
    stream.synchronize()
    return e0.elapsed_time(e1) / iters


def _time_graph(torch, stream, fn, iters, replays=5):
    """Average device time of one call of `fn`, with `iters` calls captured into one CUDA graph so
    that host launch overhead (several microseconds per call through Python) is out of the picture."""
    g = torch.cuda.CUDAGraph()
    stream.synchronize()
    with torch.cuda.graph(g, stream=stream):
        for i in range(iters):
            fn(i)
    g.replay()
    stream.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record(stream)
    for _ in range(replays):
        g.replay()
    e1.record(stream)
    stream.synchronize()
    return e0.elapsed_time(e1) / (replays * iters)


def gemv_sweep(dev, torch, stream):
    """The smaller (K,N) pairs of the GEMV sweep.  They fit in L2 (126 MB), so each is timed twice:
    'cold' rotates through enough distinct weight copies to exceed 2x L2 between reuses, 'warm'
    re-reads one copy (L2 resident)."""
    from ratchet_b200 import capi
    peak, _ = measured_peak()
    out = []
    for K, N in SWEEP_SHAPES:
        wq = make_weights(N, K, seed=K + N)
        copies = max(2, int(300e6 // wq.nbytes) + 1)
        bufs = [dev.from_quantized(wq, capi.Q8_0F, (N, K)) for _ in range(copies)]
        x = dev.from_numpy(np.random.Generator(np.random.PCG64(3)).standard_normal((1, K)).astype(np.float16))
        y = dev.empty(capi.F16, (1, N))
        run = lambda i: dev.matmul(bufs[i % copies], x, None, False, True, True, out=y)
        for i in range(copies):
            run(i)
        cold_ms = _time_graph(torch, stream, run, copies * 8)
        warm_ms = _time_graph(torch, stream, lambda i: run(0), 100)
        b = gemv_bytes(N, K)
        out.append({"K": K, "N": N, "bytes": b, "cold_us": cold_ms * 1e3, "cold_gbs": b / cold_ms / 1e6, "cold_frac_of_measured": b / cold_ms / 1e6 / peak,
                    "warm_us": warm_ms * 1e3, "warm_gbs": b / warm_ms / 1e6, "weight_copies_rotated": copies})
        for bf in bufs:
            bf.free()
    return out


def _q4kh_weights(N, K, seed):
    """Random ratchet Q4_KH buffer (dtype/blocks.rs:124-148): random nibbles and 6-bit scale/min codes,
    f16 super-block d / dmin of the magnitude an N(0, 0.02) weight produces."""
    from ratchet_b200 import capi
    rng = np.random.Generator(np.random.PCG64(seed))
    n = N * K
    nb = n // 256
    off = capi.dtype_segments(capi.Q4_KH, n)
    buf = np.zeros(capi.dtype_nbytes(capi.Q4_KH, n), np.uint8)
    buf[off[0]: off[0] + n // 2] = rng.integers(0, 256, n // 2, dtype=np.uint8)
    buf[off[1]: off[1] + nb * 12] = rng.integers(0, 256, nb * 12, dtype=np.uint8)
    buf[off[2]: off[2] + nb * 2] = np.full(nb, 0.0011, np.float16).view(np.uint8)
    buf[off[3]: off[3] + nb * 2] = np.full(nb, 0.00015, np.float16).view(np.uint8)
    return buf


def prefill_gemm_bench(dev, torch, stream):
    """Config 3: x [M, 3072] f16 . W[8192, 3072]^T with W in ratchet Q4_KH, out [M, 8192] f16, M in
    {128, 512, 2048}, timed from a CUDA graph: up to M = 512 one tcgen05 kernel that converts the Q4_K tiles
    in shared memory; beyond, a dequantise-to-f16 kernel into pooled scratch followed by the f16 tcgen05 GEMM
    (timed together).  Also the GEMM alone on f16 weights (tensor-pipe figure)."""
    from ratchet_b200 import capi
    N, K = 8192, 3072
    wq = dev.from_quantized(_q4kh_weights(N, K, 21), capi.Q4_KH, (N, K))
    wf = dev.dequantize(wq)
    peak_tf = 1678.2
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        with open(p) as f:
            peak_tf = float(json.load(f)["bf16_tflops"])
    out = []
    for M in (128, 512, 2048):
        x = dev.from_numpy(np.random.Generator(np.random.PCG64(M)).standard_normal((M, K)).astype(np.float16))
        y = dev.empty(capi.F16, (M, N))
        run_q = lambda i: dev.matmul(wq, x, None, False, True, True, out=y)
        run_f = lambda i: dev.matmul(wf, x, None, False, True, True, out=y)
        run_q(0); run_f(0)
        ms_q = _time_graph(torch, stream, run_q, 20)
        ms_f = _time_graph(torch, stream, run_f, 20)
        flops = 2.0 * M * N * K
        out.append({"M": M, "N": N, "K": K, "q4k_us": ms_q * 1e3, "q4k_tflops": flops / ms_q / 1e9, "f16_gemm_us": ms_f * 1e3,
                    "f16_gemm_tflops": flops / ms_f / 1e9, "f16_gemm_frac_of_measured_bf16_peak": flops / ms_f / 1e9 / peak_tf,
                    "bytes": M * K * 2 + 14155776 + M * N * 2})
    return out


PHI3 = dict(n_layers=32, d=3072, n_heads=32, head_dim=96, ffn=8192, vocab=32064, max_cache=4096, kv_prior=1024)


def _q8h_weights(N, K, seed):
    """Q8_0H buffer (f16 scales) with random int8 codes and scales of N(0,0.02)-like magnitude.  Built
    directly in the quantised domain: the decode benchmark needs the bytes, not a float original."""
    from ratchet_b200 import capi
    rng = np.random.Generator(np.random.PCG64(seed))
    buf = np.zeros(capi.dtype_nbytes(capi.Q8_0H, N * K), np.uint8)
    uniq = min(N, 1024)
    q = rng.integers(-127, 128, (uniq, K), dtype=np.int8)
    d = (np.abs(rng.standard_normal((uniq, K // 32))) * 0.0004 + 0.0003).astype(np.float16)
    qs = buf[: N * K].view(np.int8).reshape(N, K)
    off = capi.dtype_segments(capi.Q8_0H, N * K)[1]
    ds = buf[off: off + (N * K // 32) * 2].view(np.float16).reshape(N, K // 32)
    for r0 in range(0, N, uniq):
        r1 = min(N, r0 + uniq)
        qs[r0:r1] = q[: r1 - r0]
        ds[r0:r1] = d[: r1 - r0]
    return buf


def _lazy_forward_us(torch, stream, build_and_resolve, iters):
    """Average time of one forward through the lazy Tensor API (graph build on the host + resolve on the
    device), CUDA events on the library's stream around `iters` forwards after three warm-ups."""
    for _ in range(3):
        build_and_resolve()
    stream.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record(stream)
    for _ in range(iters):
        build_and_resolve()
    e1.record(stream)
    stream.synchronize()
    return e0.elapsed_time(e1) * 1e3 / iters


def _lazy_forward_device_us(torch, stream, build_and_resolve, iters):
    """Device time of the same forward with the host out of the picture: the launches of one build + resolve
    are captured into a CUDA graph (the resolver neither synchronises nor allocates from the driver once its
    pool is warm) and the graph is replayed.  None if the capture is refused."""
    try:
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph, stream=stream):
            keep = build_and_resolve()       # alive until the capture ends
        del keep
        graph.replay()
        stream.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record(stream)
        for _ in range(iters):
            graph.replay()
        e1.record(stream)
        stream.synchronize()
        return e0.elapsed_time(e1) * 1e3 / iters
    except Exception:
        return None


def phi2_mlp_bench(dev, torch, stream):
    """Config 1: Phi-2 MLP block in f32 through the lazy Tensor graph: x [1,64,2560] N(0,1), LayerNorm,
    W1 [10240,2560] + b1, tanh-GELU, W2 [2560,10240] + b2, residual.  HBM-bound at M=64 (210 MB of weights)."""
    from ratchet_b200 import Tensor, callers, nn
    g = np.random.Generator(np.random.PCG64(0))
    d, ffn = 2560, 10240
    t = lambda a: Tensor.from_data(a, device=dev)
    x = t(g.standard_normal((1, 64, d), dtype=np.float32))
    blk = callers.Phi2MLPBlock(nn.LayerNorm(t(np.ones(d, np.float32)), t(np.zeros(d, np.float32)), 1e-5),
                               nn.Linear(t(g.standard_normal((ffn, d), dtype=np.float32) * np.float32(0.02)), t(np.zeros(ffn, np.float32))),
                               nn.Linear(t(g.standard_normal((d, ffn), dtype=np.float32) * np.float32(0.02)), t(np.zeros(d, np.float32))))
    us = _lazy_forward_us(torch, stream, lambda: blk.schedule(x).resolve(), 50)
    dev_us = _lazy_forward_device_us(torch, stream, lambda: blk.schedule(x).resolve(), 50)
    nbytes = 2 * ffn * d * 4 + 4 * 64 * d * 4
    flops = 2.0 * 64 * d * ffn * 2
    peak, kind = measured_peak()
    return {"us_per_forward": us, "device_us_per_forward": dev_us, "algorithmic_bytes": nbytes, "gbs": nbytes / us * 1e-3, "frac_of_hbm_peak": nbytes / us * 1e-3 / peak,
            "peak_kind": f"of {kind}", "tflops": flops / us * 1e-6, "note": "weights (210 MB) exceed L2; lazy graph build + resolve each forward"}


def _q8f_random(N, K, seed):
    """Q8_0F buffer (f32 scales) of random int8 codes with scales that give weights of N(0, 0.02)-like size."""
    from ratchet_b200 import capi
    rng = np.random.Generator(np.random.PCG64(seed))
    buf = np.zeros(capi.dtype_nbytes(capi.Q8_0F, N * K), np.uint8)
    buf[: N * K].view(np.int8)[:] = rng.integers(-127, 128, N * K, dtype=np.int8)
    off = capi.dtype_segments(capi.Q8_0F, N * K)[1]
    buf[off: off + (N * K // 32) * 4].view(np.float32)[:] = (np.abs(rng.standard_normal(N * K // 32)) * 0.0002 + 0.0003).astype(np.float32)
    return buf


def _q8h_random(N, K, seed):
    """Q8_0H buffer (f16 scales) of random int8 codes with scales that give weights of N(0, 0.02)-like size."""
    from ratchet_b200 import capi
    rng = np.random.Generator(np.random.PCG64(seed))
    buf = np.zeros(capi.dtype_nbytes(capi.Q8_0H, N * K), np.uint8)
    buf[: N * K].view(np.int8)[:] = rng.integers(-127, 128, N * K, dtype=np.int8)
    off = capi.dtype_segments(capi.Q8_0H, N * K)[1]
    buf[off: off + (N * K // 32) * 2].view(np.float16)[:] = (np.abs(rng.standard_normal(N * K // 32)) * 0.0002 + 0.0003).astype(np.float16)
    return buf


def whisper_encoder_bench(dev, torch, stream, mode="f32"):
    """Config 4: Whisper-tiny encoder forward through the lazy Tensor graph: mel [1,80,3000] U(-1,1),
    conv stem, sinusoidal positions, 4 pre-LN blocks (d 384, 6 heads, MLP 1536), final LayerNorm.
    mode "f32": f32 activations and weights N(0, 0.02); "q8f": f32 activations, Linear weights as Q8_0F
    buffers; "q8h": f16 activations and parameters, Linear weights as Q8_0H buffers (what ratchet loads on
    a device with f16 support)."""
    from ratchet_b200 import Tensor, callers, capi, nn
    g = np.random.Generator(np.random.PCG64(0))
    d, H, mlp, n_ctx = 384, 6, 1536, 1500
    seeds = iter(range(1000, 2000))
    quantised = mode != "f32"
    act_np, act_dt = (np.float16, capi.F16) if mode == "q8h" else (np.float32, capi.F32)

    def w(*shape):
        if quantised and len(shape) == 2:
            return None, shape
        return g.standard_normal(shape, dtype=np.float32) * np.float32(0.02)

    def t(a):   # Linear weights come as (None, shape) when they are to be quantised
        if isinstance(a, tuple):
            if mode == "q8h":
                return Tensor.from_quantized(_q8h_random(a[1][0], a[1][1], next(seeds)), capi.Q8_0H, a[1], dev)
            return Tensor.from_quantized(_q8f_random(a[1][0], a[1][1], next(seeds)), capi.Q8_0F, a[1], dev)
        return Tensor.from_data(np.ascontiguousarray(a, np.float32), device=dev)    # parameters stay f32, as the checkpoint has them
    inc = np.log(10000.0) / (d // 2 - 1)
    ang = np.arange(n_ctx)[:, None] * np.exp(-inc * np.arange(d // 2))[None, :]
    pos = np.concatenate([np.sin(ang), np.cos(ang)], 1)
    dk = Tensor.from_data(np.array([np.float32(d // H) ** np.float32(-0.25)], np.float32).astype(act_np), device=dev)
    blocks = []
    for _ in range(4):
        mha = callers.WhisperMHA(nn.Linear(t(w(d, d)), t(w(d))), nn.Linear(t(w(d, d)), None), nn.Linear(t(w(d, d)), t(w(d))),
                                 nn.Linear(t(w(d, d)), t(w(d))), H, dk)
        blocks.append(callers.WhisperBlock(nn.LayerNorm(t(np.ones(d)), t(np.zeros(d)), 1e-5), mha,
                                           nn.LayerNorm(t(np.ones(d)), t(np.zeros(d)), 1e-5),
                                           callers.WhisperMLP(nn.Linear(t(w(mlp, d)), t(w(mlp))), nn.Linear(t(w(d, mlp)), t(w(d))))))
    enc = callers.WhisperEncoder(t(w(d, 80, 3)), t(w(d)), t(w(d, d, 3)), t(w(d)), t(pos), blocks,
                                 nn.LayerNorm(t(np.ones(d)), t(np.zeros(d)), 1e-5), act_dt)
    mel = t(g.uniform(-1.0, 1.0, (1, 80, 3000)))
    l0 = dev.launches
    enc.schedule(mel).resolve()
    launches = dev.launches - l0
    us = _lazy_forward_us(torch, stream, lambda: enc.schedule(mel).resolve(), 20)
    dev_us = _lazy_forward_device_us(torch, stream, lambda: enc.schedule(mel).resolve(), 20)
    # flops: conv stem + per block (4 projections, QK^T, PV, two MLP matmuls)
    flops = 2.0 * 3000 * d * 80 * 3 + 2.0 * n_ctx * d * d * 3 + 4 * (2.0 * n_ctx * d * d * 4 + 2 * 2.0 * n_ctx * n_ctx * d + 2 * 2.0 * n_ctx * d * mlp)
    what = {"f32": "f32 activations and weights",
            "q8f": "f32 activations, Q8_0F Linear weights (dequantised into pooled scratch, then the f32 tensor-core GEMM)",
            "q8h": "f16 activations, Q8_0H Linear weights (tcgen05 f16 GEMM)"}[mode]
    score_mb = 6 * n_ctx * n_ctx * (2 if mode == "q8h" else 4) * 3 / 1e6
    return {"us_per_forward": us, "device_us_per_forward": dev_us, "kernels_per_forward": int(launches), "tflops": flops / us * 1e-6,
            "note": what + f"; mixed launch- and compute-bound ({score_mb:.0f} MB of 1500x1500 score matrices per layer pass through L2)"}


def phi3_decode_bytes(c):
    """Algorithmic HBM bytes of one decode step: Q8_0H weights (1 + 2/32 bytes per element) of every
    Linear + one embedding row, K and V rows of the populated cache, negligible activations."""
    d, ffn, V, L = c["d"], c["ffn"], c["vocab"], c["n_layers"]
    w_elems = L * (3 * d * d + d * d + 2 * ffn * d + d * ffn) + V * d
    kv = L * 2 * c["n_heads"] * (c["kv_prior"] + 1) * c["head_dim"] * 2
    return int(w_elems * (1 + 2 / 32)) + kv + d * (1 + 2 / 32)


def phi3_decode_bench(dev, torch, stream, steps, warmup, rank=0, world=1, dist=None):
    """Phi-3-mini decode step (32 layers, hidden 3072, 32 heads x 96, MLP 8192, vocab 32064, Q8_0H
    weights, 1024 prior KV positions of N(0,1) f16, batch 1) through the fused decode engine.  With
    world > 1 every Linear is sharded by output rows over the ranks (attention by heads) and each rank
    holds its own rows, generated at the shard's shape: the weights are random either way."""
    from ratchet_b200 import capi
    from ratchet_b200.decoder import Decoder, DecoderConfig, DecoderLayer
    c = PHI3
    d, H, hd, ffn, V = c["d"], c["n_heads"], c["head_dim"], c["ffn"], c["vocab"]
    g = world
    Hl = H // g
    rng = np.random.Generator(np.random.PCG64(11))
    shapes = {"qkv": (3 * Hl * hd, d), "o": (d // g, d), "up": (2 * ffn // g, d), "down": (d // g, ffn)}
    host = {k: _q8h_weights(n, kk, 100 * rank + i) for i, (k, (n, kk)) in enumerate(shapes.items())}
    kv_host = np.zeros((Hl, c["max_cache"], hd), np.float16)
    kv_host[:, : c["kv_prior"]] = rng.standard_normal((Hl, c["kv_prior"], hd)).astype(np.float16)
    ones = np.ones(d, np.float32)
    layers = []
    for _ in range(c["n_layers"]):   # every layer gets its own device copy: the step streams 32 distinct sets
        layers.append(DecoderLayer(dev.from_numpy(ones), dev.from_quantized(host["qkv"], capi.Q8_0H, shapes["qkv"]),
                                   dev.from_quantized(host["o"], capi.Q8_0H, shapes["o"]), dev.from_numpy(ones),
                                   dev.from_quantized(host["up"], capi.Q8_0H, shapes["up"]), dev.from_quantized(host["down"], capi.Q8_0H, shapes["down"]),
                                   dev.from_numpy(kv_host), dev.from_numpy(kv_host)))
    emb = dev.from_quantized(_q8h_weights(V, d, 5), capi.Q8_0H, (V, d))          # same table on every rank
    head = dev.from_quantized(_q8h_weights(V // g, d, 6 + rank), capi.Q8_0H, (V // g, d))
    cfg = DecoderConfig(c["n_layers"], d, H, H, hd, ffn, V, c["max_cache"], hd, 10000.0, 1e-5, capi.Q8_0H)
    comm = None
    if world > 1:
        from ratchet_b200.comm import Comm
        comm = Comm(dev, rank, world, max(d, ffn, V, H * hd), bytes_per_elem=4)
    dec = Decoder(dev, cfg, layers, emb, dev.from_numpy(ones), head, comm=comm)

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    tok_host = torch.tensor([int(rng.integers(0, V))], dtype=torch.int32).pin_memory()
    tok_dev = torch.empty(1, dtype=torch.int32, device="cuda")
    tok_dev.copy_(tok_host)
    logits_host = torch.empty(V, dtype=torch.float16).pin_memory()
    logits_dev = torch.empty(V, dtype=torch.float16, device="cuda")
    import ctypes as C

    def step(_i=0):
        dec.position = c["kv_prior"]          # keep the workload fixed: 1024 prior positions every step
        dev.check(dev._lib.rcu_decoder_step(dec._h, C.c_void_p(tok_dev.data_ptr()), C.c_void_p(logits_dev.data_ptr()), None))

    def step_e2e(_i=0):
        tok_dev.copy_(tok_host, non_blocking=True)     # ids up (phi3/generate.rs:95-96)
        step()
        logits_host.copy_(logits_dev, non_blocking=True)   # logits down, arg-max on the host (generate.rs:101-108)
        stream.synchronize()
        tok_host[0] = int(torch.argmax(logits_host.float()))

    for _ in range(warmup):
        step()
    barrier()
    job_profile = None
    if world == 1 and os.environ.get("RCU_BENCH_JOB_PROFILE"):
        # per-job time table of the data-flow kernel (device time stamps of its first CTA), median of five steps
        runs = []
        for _ in range(5):
            dec.position = c["kv_prior"]
            raw = dec.profile_step(tok_dev.data_ptr()).astype(np.int64)
            cyc = raw[-24:].reshape(6, 4)
            runs.append(np.diff(raw[:-24]))
        med = np.median(np.stack(runs), 0)           # [stage, work] per job
        names = ["qkv", "attention", "o", "gate_up", "down"]
        per_layer = med[: 10 * c["n_layers"]].reshape(c["n_layers"], 5, 2)
        job_profile = {"us_per_layer_median": {n: {"input_wait_and_stage": float(np.median(per_layer[:, i, 0])) / 1e3,
                                                   "items_and_tail": float(np.median(per_layer[:, i, 1])) / 1e3} for i, n in enumerate(names)},
                       "layer_us_median": float(np.median(per_layer.sum((1, 2)))) / 1e3,
                       "lm_head_us": float(med[-2:].sum()) / 1e3, "kernel_us": float(med.sum()) / 1e3,
                       "first_warp_cycles_per_step": {k: dict(zip(["slot_wait", "multiply", "store", "request"], [int(v) for v in cyc[i]]))
                                                      for i, k in enumerate(["qkv", "attention", "o", "gate_up", "down", "lm_head"])}}
    l0 = dev.launches
    ms = _time_loop(torch, stream, step, steps)
    launches = (dev.launches - l0) // steps
    barrier()
    for _ in range(3):
        step_e2e()
    barrier()
    t0 = time.perf_counter()
    for _ in range(steps):
        step_e2e()
    barrier()
    e2e_s = (time.perf_counter() - t0) / steps
    dev.sync()     # a flag wait that ran out of time surfaces here
    if world > 1:
        t = torch.tensor([ms, e2e_s], dtype=torch.float64, device="cuda")
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        ms, e2e_s = (float(v) for v in t.tolist())
    b = phi3_decode_bytes(c)            # whole model; each rank streams 1/world of the Linear weights and KV
    peak, kind = measured_peak()
    res = {"metric": "phi3_mini_q8_0_decode_tokens_per_s", "value": 1e3 / ms, "unit": "tokens/s", "n_gpus": world, "ms_per_token": ms,
           "e2e_tokens_per_s": 1.0 / e2e_s, "h2d_bytes_per_step": 4, "d2h_bytes_per_step": V * 2,
           "kernels_per_token": int(launches), "algorithmic_bytes_per_token": b, "achieved_gbs": b / ms / 1e6,
           "roofline_frac": b / ms / 1e6 / (peak * world), "roofline_tokens_per_s": world * peak * 1e9 / b, "peak_kind": f"of {kind}",
           "parallelism": "single GPU" if world == 1 else f"every Linear row-sharded x{world}, attention by heads, 4 fused all-gathers per layer (peer stores over NVLink)",
           "config": {"model": "phi-3-mini shape, random Q8_0H weights", **c, "steps": steps}}
    if job_profile is not None:
        res["job_profile"] = job_profile
    dec.close()
    if comm is not None:
        dist.barrier()
        comm.close()
    return res


def sharded_decode_check(dev, torch, rank, world, dist):
    """Two Phi-3-mini layers at full width, three greedy steps: the sharded decoder's logits against the
    single-GPU decoder's on every rank.  Each output element is computed by one rank with the single-GPU
    arithmetic, so where both take the same kernels (up to four ranks) the logits are equal bit for bit; on
    eight ranks the sharded step runs one kernel per phase, whose GEMVs sum in another order, and the
    comparison is the quantised-matmul bar (1e-2 of the logits' scale).  Run outside every timed region."""
    from ratchet_b200 import capi
    from ratchet_b200.comm import Comm, decoder_shard_ranges, take_rows_q8
    from ratchet_b200.decoder import Decoder, DecoderConfig, DecoderLayer
    c = PHI3
    d, H, hd, ffn, V, L, prior, cache = c["d"], c["n_heads"], c["head_dim"], c["ffn"], c["vocab"], 2, c["kv_prior"], 2048
    R = decoder_shard_ranges(H, H, hd, d, ffn, V, rank, world)
    rows = lambda key: sum(b - a for a, b in R[key])
    rng = np.random.Generator(np.random.PCG64(77))
    ones = np.ones(d, np.float32)
    full = {"qkv": (3 * d, d), "o": (d, d), "gate_up": (2 * ffn, d), "down": (d, ffn)}
    host = [{k: _q8h_weights(n, kk, 900 + 10 * li + i) for i, (k, (n, kk)) in enumerate(full.items())} for li in range(L)]
    kv = rng.standard_normal((L, 2, H, prior, hd)).astype(np.float16)
    emb_h, head_h = _q8h_weights(V, d, 990), _q8h_weights(V, d, 991)
    h0, h1 = R["kv_heads"]

    def build(sharded, comm):
        layers = []
        for li in range(L):
            w = {}
            for k, (n, kk) in full.items():
                if sharded:
                    w[k] = dev.from_quantized(take_rows_q8(host[li][k], capi.Q8_0H, n, kk, R[k]), capi.Q8_0H, (rows(k), kk))
                else:
                    w[k] = dev.from_quantized(host[li][k], capi.Q8_0H, (n, kk))
            heads = slice(h0, h1) if sharded else slice(0, H)
            kc = np.zeros((heads.stop - heads.start, cache, hd), np.float16)
            vc = np.zeros_like(kc)
            kc[:, :prior] = kv[li, 0, heads]
            vc[:, :prior] = kv[li, 1, heads]
            layers.append(DecoderLayer(dev.from_numpy(ones), w["qkv"], w["o"], dev.from_numpy(ones), w["gate_up"], w["down"],
                                       dev.from_numpy(kc), dev.from_numpy(vc)))
        head = dev.from_quantized(take_rows_q8(head_h, capi.Q8_0H, V, d, R["lm_head"]), capi.Q8_0H, (rows("lm_head"), d)) if sharded \
            else dev.from_quantized(head_h, capi.Q8_0H, (V, d))
        cfg = DecoderConfig(L, d, H, H, hd, ffn, V, cache, hd, 10000.0, 1e-5, capi.Q8_0H)
        dec = Decoder(dev, cfg, layers, dev.from_quantized(emb_h, capi.Q8_0H, (V, d)), dev.from_numpy(ones), head, comm=comm)
        dec.position = prior
        return dec

    def run(dec):
        out = []
        dev.h2d(dec.token.ptr, np.array([1234], np.int32))
        for i in range(3):
            dec.step_device(dec.token.ptr if i == 0 else dec.next_token.ptr)
            dev.sync()
            out.append(dec.logits.to_numpy().copy())
        return out

    single = build(False, None)
    ref = run(single)
    single.close()
    comm = Comm(dev, rank, world, max(d, ffn, V, H * hd), bytes_per_elem=4)
    shard = build(True, comm)
    got = run(shard)
    same = all(np.array_equal(a.view(np.uint16), b.view(np.uint16)) for a, b in zip(got, ref))
    rel = max(float(np.abs(a.astype(np.float32) - b.astype(np.float32)).max() / np.sqrt(np.mean(b.astype(np.float32) ** 2))) for a, b in zip(got, ref))
    flag = torch.tensor([1 if same else 0], dtype=torch.int32, device="cuda")
    dist.all_reduce(flag, op=dist.ReduceOp.MIN)
    worst = torch.tensor([rel], dtype=torch.float64, device="cuda")
    dist.all_reduce(worst, op=dist.ReduceOp.MAX)
    dist.barrier()
    shard.close()
    comm.close()
    return {"sharded_logits_equal_single_gpu_bits": bool(int(flag.item())), "max_abs_diff_over_rms": float(worst.item()),
            "within_1e-2": bool(float(worst.item()) <= 1e-2), "layers": L, "steps": 3, "ranks": world}


def run_ours(args):
    import torch
    import torch.distributed as dist

    from ratchet_b200 import Device, capi

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if not torch.cuda.is_available():
        raise SystemExit("bench.py needs a CUDA device: the CUDA library has no CPU fallback")
    torch.cuda.set_device(local_rank)
    if world > 1:
        dist.init_process_group("nccl", device_id=torch.device("cuda", local_rank))
    # a stream of our own: CUDA-graph capture (used by the decode engine) is not allowed on the legacy default stream
    stream = torch.cuda.Stream()
    torch.cuda.set_stream(stream)
    dev = Device(local_rank, stream=stream.cuda_stream)
    # every weight matrix of this benchmark is uploaded once and never written again, as a loaded model's are: say so,
    # so that GEMVs launched back to back may start fetching weights while their predecessor drains
    dev.set_constant_weights(True)

    K, N = K_HEAD, (args.rows or N_HEAD)
    n_local = N // world
    wq = make_weights(n_local, K, seed=1000)      # every shard is the same 4096 rows repeated (n_local is a multiple of 4096 up to 8 GPUs)
    dw = dev.from_quantized(wq, capi.Q8_0F, (n_local, K))
    del wq
    rng = np.random.Generator(np.random.PCG64(7))
    x_host = torch.from_numpy(rng.standard_normal((1, K)).astype(np.float16)).pin_memory()
    x_dev = torch.empty((1, K), dtype=torch.float16, device="cuda")
    x_dev.copy_(x_host)
    y_full = torch.empty((1, N), dtype=torch.float16, device="cuda")      # gathered output
    y_local = y_full[:, rank * n_local:(rank + 1) * n_local] if world == 1 else torch.empty((1, n_local), dtype=torch.float16, device="cuda")
    y_host = torch.empty((2, N), dtype=torch.float16).pin_memory()          # results of two steps in flight
    bx = dev.wrap(capi.F16, (1, K), x_dev.data_ptr())
    by = dev.wrap(capi.F16, (1, n_local), y_local.data_ptr())
    y_alt = torch.empty((1, n_local), dtype=torch.float16, device="cuda")    # N = 1: second output buffer for the end-to-end loop
    by_alt = dev.wrap(capi.F16, (1, n_local), y_alt.data_ptr())
    # a second handle of the library on a stream of its own carries the device-to-host copies, so that the copy of
    # one step's result overlaps the next step's kernel
    copy_stream = torch.cuda.Stream()
    dev_copy = Device(local_rank, stream=copy_stream.cuda_stream)

    comm = None
    if world > 1:
        # one window per rank; torch.distributed only carries the 64-byte IPC handles (plumbing)
        from ratchet_b200.comm import Comm
        comm = Comm(dev, rank, world, N)
    y_host_np = y_host.numpy()

    def step():
        if comm is None:
            dev.matmul(dw, bx, None, False, True, True, out=by)
            return None
        # local GEMV whose last CTA pushes the slice to every peer over NVLink, then a bounded flag wait
        return comm.linear(dw, bx, N)

    x_host_np = x_host.numpy()

    def step_e2e(i):
        # Host buffers in and out through the C ABI, every step: rcu_h2d of the activation (pinned source), the
        # GEMV, and rcu_d2h_async of the whole result on the copy handle behind rcu_stream_wait.  The kernel of
        # step i + 2 is ordered after the copy of step i: the gathered output rotates through three slots (two
        # buffers at N = 1), so a slot is never rewritten while its copy is in flight.
        if i >= 2:
            dev.wait_for(dev_copy)             # copies up to step i - 1 are queued there; the copy of step i - 2 is what matters
        dev.h2d(bx.ptr, x_host_np, K * 2)
        if comm is None:
            out = by if i % 2 == 0 else by_alt
            dev.matmul(dw, bx, None, False, True, True, out=out)
        else:
            out = comm.linear(dw, bx, N)
        dev_copy.wait_for(dev)
        dev_copy.d2h_async(y_host_np[i % 2], out.ptr, N * 2)

    def run_e2e(n):
        for i in range(n):
            step_e2e(i)
        dev_copy.sync()
        dev.sync()

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    for _ in range(max(args.warmup, 3)):
        step()
    barrier()
    sampler = ClockSampler(local_rank)
    if rank == 0:
        sampler.start()
    launches0 = dev.launches
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    graph = None
    if world > 1:
        # the K steps as one captured CUDA graph: eight Python processes launching step by step would put
        # their host skew inside every step's peer wait
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph, stream=stream):
            for _ in range(args.steps):
                step()
        barrier()
        graph.replay()                      # one untimed replay: first-use costs of the instantiated graph
    barrier()
    mark0 = sampler.mark()
    ev0.record(stream)
    if graph is not None:
        graph.replay()
    else:
        for _ in range(args.steps):
            step()
    ev1.record(stream)
    barrier()
    mark1 = sampler.mark()
    ms = ev0.elapsed_time(ev1)
    launches = (dev.launches - launches0) if graph is None else args.steps
    # Every step is exactly one launch of the GEMV kernel (at N > 1 the same kernel also pushes its slice to
    # the peers and waits for theirs), so the kernel's average launch duration is the timed region / steps.
    kernel_ms = ms / args.steps
    # end to end: host activation in, host result out, every step
    run_e2e(4)
    barrier()
    t0 = time.perf_counter()
    run_e2e(args.steps)
    barrier()
    e2e_s = (time.perf_counter() - t0) / args.steps

    # The collective this fused gather replaces, on the same box: the plain GEMV into a local buffer, then
    # torch.distributed's NCCL all-gather of the f16 slices (a reported comparison, not the product path).
    nccl = None
    if world > 1:
        y_gather = torch.empty((1, N), dtype=torch.float16, device="cuda")

        def step_nccl():
            dev.matmul(dw, bx, None, False, True, True, out=by)
            dist.all_gather_into_tensor(y_gather, y_local)
        for _ in range(5):
            step_nccl()
        barrier()
        n0, n1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        n0.record(stream)
        for _ in range(args.steps):
            step_nccl()
        n1.record(stream)
        barrier()
        nccl_ms = n0.elapsed_time(n1) / args.steps
    clocks = sampler.stop(mark0, max(mark1, mark0 + 1)) if rank == 0 else None

    # What was timed is checked, outside the timed region: one more step, the gathered output of all ranks
    # against the oracle on the 4096 distinct rows (every row of every shard repeats one of them).
    parity = None
    out = step()
    dev.sync()
    y_all = np.empty(N, np.float16)
    dev.d2h(y_all, by.ptr if out is None else out.ptr, N * 2)
    if rank == 0:
        from oracle import oracle as orc
        uniq = min(n_local, UNIQUE_ROWS)
        ref = orc.gemv_q8(orc.quantize_q8(unique_rows(K, 1000)[:uniq]), uniq, K, False, x_host_np.reshape(-1)).astype(np.float32)
        ref_all = np.tile(ref, N // uniq + 1)[:N] if n_local % uniq == 0 else None
        if ref_all is not None:
            parity = parity_report(y_all.astype(np.float32), ref_all, rtol=1e-2, atol=1e-2 * float(np.sqrt(np.mean(ref * ref))))
            parity["against"] = "CPU oracle (dequantise + f32 matmul), every output row of every rank"

    t = torch.tensor([ms, kernel_ms, e2e_s, nccl_ms if world > 1 else 0.0], dtype=torch.float64, device="cuda")
    if world > 1:
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
    ms, kernel_ms, e2e_s, nccl_ms = (float(v) for v in t.tolist())
    ms_per_step = ms / args.steps
    total_bytes = gemv_bytes(N, K)
    value = total_bytes / (ms_per_step * 1e-3) / 1e9
    peak, peak_kind = measured_peak()
    local_bytes = gemv_bytes(n_local, K)
    achieved = local_bytes / (kernel_ms * 1e-3) / 1e9

    line = {}
    if rank == 0:
        line = {
            "metric": "q8_0_gemv_gbs", "value": value, "unit": "GB/s", "n_gpus": world, "steps": args.steps, "warmup": max(args.warmup, 3),
            "ms_per_step": ms_per_step, "higher_is_better": True, "scaling": "strong", "vs_baseline": None,
            "dtype": "i8xf16->f32", "data": "synthetic",
            "config": {"workload": WORKLOAD, "K": K, "N": N, "rows_per_gpu": n_local, "parallelism": f"row-shard x{world}, all-gather fused into the GEMV (peer stores over NVLink)" if world > 1 else "single GPU",
                       "l2": "weights per GPU exceed L2 (126 MB) at every N <= 8; no flush"},
            "e2e": {"value": total_bytes / e2e_s / 1e9, "unit": "GB/s", "h2d_bytes_per_step": K * 2, "d2h_bytes_per_step": N * 2,
                    "note": "weights stay resident (loaded once, as ratchet loads a model); activation rcu_h2d and result rcu_d2h_async every step, "
                            "the copy of step i overlapping the kernel of step i + 1 (second library handle on a copy stream)"},
            "gpu_launches": int(launches),
            "parity": parity,
            "clocks": clocks,
            "roofline": {"bound": "hbm", "achieved": achieved, "peak": peak, "unit": "GB/s", "frac": achieved / peak,
                         "peak_kind": f"of {peak_kind}", "frac_of_nominal_8TBs": achieved / 8000.0, "kernel": "gemv_q8_ring_kernel",
                         "kernel_ms": kernel_ms, "bytes_per_launch": local_bytes, "traffic": None},
        }
        line["roofline"]["traffic"] = GEMV_TRAFFIC_PER_ROW_BYTES * n_local
        if world > 1:
            line["nccl_allgather_baseline"] = {"ms_per_step": nccl_ms, "gbs": total_bytes / (nccl_ms * 1e-3) / 1e9,
                                               "what": "plain GEMV on the shard + torch.distributed all_gather_into_tensor (NCCL) of the f16 slices, same stream, un-graphed"}
        if world == 1 and not args.rows:
            line["cpu_baseline"] = cpu_baseline_sample(K, N)
    # release the GEMV weights before the other legs allocate theirs
    del dw
    extras = {}
    legs = set(args.legs.split(","))
    want = lambda name: "all" in legs or name in legs
    if world == 1 and not args.rows and not args.no_extras:
        if want("sweep"):
            extras["gemv_sweep"] = gemv_sweep(dev, torch, stream)
        if want("prefill"):
            extras["q4k_prefill_gemm"] = prefill_gemm_bench(dev, torch, stream)
        if want("phi2"):
            extras["phi2_mlp_f32"] = phi2_mlp_bench(dev, torch, stream)
        if want("whisper"):
            extras["whisper_tiny_encoder_f32"] = whisper_encoder_bench(dev, torch, stream)
            extras["whisper_tiny_encoder_q8_0f"] = whisper_encoder_bench(dev, torch, stream, mode="q8f")
            extras["whisper_tiny_encoder_q8_0h"] = whisper_encoder_bench(dev, torch, stream, mode="q8h")
        if want("decode"):
            extras["phi3_decode"] = phi3_decode_bench(dev, torch, stream, steps=min(args.steps, 200), warmup=max(args.warmup, 3))
    if world > 1 and not args.rows and not args.no_extras:
        if comm is not None:            # the GEMV leg's window goes first: one exchange window per rank at a time
            dist.barrier()
            comm.close()
            comm = None
        check = sharded_decode_check(dev, torch, rank, world, dist)
        extras["phi3_decode"] = phi3_decode_bench(dev, torch, stream, steps=min(args.steps, 200), warmup=max(args.warmup, 3), rank=rank,
                                                  world=world, dist=dist)
        extras["phi3_decode"]["parity"] = check
    if rank == 0:
        line.update(extras)
        print(json.dumps(line))
    if comm is not None:
        dist.barrier()
        comm.close()
    dev_copy.close()
    dev.close()
    if world > 1:
        dist.destroy_process_group()


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=500)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--rows", type=int, default=0,
                    help="profiling aid: run the same GEMV with this many rows instead of 65536 (no CPU baseline); "
                         "8192 rows = 134 MB of weights, still larger than L2, small enough for an ncu capture")
    ap.add_argument("--no-extras", action="store_true", help="skip the GEMV sweep and the Phi-3 decode leg")
    ap.add_argument("--legs", default="all", help="comma list of the extra legs to run at N=1: sweep, prefill, phi2, whisper, decode (default all)")
    ap.add_argument("--serve", action="store_true", help="instead: prefill and decode throughput of the Mefesun and Dadezen decoders beside Phi-3 layers of equal size")
    ap.add_argument("--serve-sizes", default="", help="with --serve: comma list of w1024, w2048, w4096 (default all)")
    ap.add_argument("--serve-models", default="", help="with --serve: comma list of mefesun, dadezen (default both)")
    ap.add_argument("--serve-only-new", action="store_true", help="with --serve: leave the Phi-3 layers out")
    args = ap.parse_args()
    if args.serve:
        from bench_serve import run_serve
        path = os.path.join(ROOT, "MEASURED_PEAKS.json")
        run_serve(args, json.load(open(path)) if os.path.exists(path) else {}, ClockSampler)
    elif args.impl == "reference":
        run_reference(args)
    else:
        run_ours(args)


if __name__ == "__main__":
    main()
