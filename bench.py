#!/usr/bin/env python
"""Headline benchmark: int4 group-32 dequant-GEMV, K=4096 -> N=14336 (Llama-3-8B FFN up-projection
shape), f16 block scales, bf16 activations, M decode tokens (default 1).

A *step* is one decode pass over LAYERS distinct weight matrices of that shape (default 32, about
1.06 GB, so every launch streams weights that are not in the 126 MB L2), replayed from one CUDA
graph.  `value` is the whole-job HBM stream rate in TB/s: algorithmic bytes (packed nibbles + f16
scales + activations in + bf16 results out) divided by device time.  With N GPUs every rank owns
its own LAYERS matrices (column-parallel shards never exchange data on this path), so scaling is
weak and the aggregate is the sum over ranks.

    python bench.py --gpus 1 --steps 50 --warmup 5
    python -m torch.distributed.run --nnodes=1 --nproc-per-node N ... bench.py --gpus N ...
    python bench.py --impl reference        # the CPU restatement of tang-infer on the host cores
    python bench.py --tofazen               # instead: the Tofazen family beside the int4 model (one JSON line of its own)
    python bench.py --numuzen               # instead: the Numuzen family beside the Tofazen family (one JSON line of its own)
    python bench.py --dotanex               # instead: the Dotanex family beside the Numuzen family (one JSON line of its own)
    python bench.py --sakinex               # instead: the Sakinex family beside the Numuzen family (one JSON line of its own)

The JSON line also carries: `e2e` (the same rate through the reference-shaped call q4_matvec with
HOST vectors, copies inside the timed region), `roofline` (dominant kernel vs measured HBM peak),
`cpu_baseline` (the oracle port on a bounded sample), `decode` (Llama-3-8B-shaped decode step,
tokens/s, when --decode is given), `clocks`, `gpu_launches`.
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

N_OUT, K_IN, GROUP = 14336, 4096, 32
METRIC, UNIT = "int4_gemv_hbm_tbps", "TB/s"

# dram__bytes_read.sum + dram__bytes_write.sum per launch of the dominant kernel, from one ncu
# capture of this command with 8 layers and 1 step (33.10 MB read; the 28 KB of results stay in L2).
NCU_TRAFFIC_BYTES_PER_LAUNCH = 33_104_640


def algorithmic_bytes(m: int) -> int:
    """Bytes one launch has to move: nibbles + f16 scales + bf16 activations in + bf16 results out."""
    return N_OUT * K_IN // 2 + N_OUT * (K_IN // GROUP) * 2 + m * K_IN * 2 + m * N_OUT * 2


def measured_peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        try:
            d = json.load(open(path))
            return float(d["hbm_gbs"]), "measured"
        except Exception:
            pass
    return 6650.0, "fallback"


class ClockSampler:
    """Samples SM clock and throttle reasons of one GPU with nvidia-smi while the timed region runs."""

    FIELDS = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
              "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_index: int):
        self.gpu_index, self.lines, self.proc, self.thread = gpu_index, [], None, None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits", "-lms", "100",
                 "-i", str(self.gpu_index)], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.proc = None
            return
        self.thread = threading.Thread(target=self._pump, daemon=True)
        self.thread.start()

    def _pump(self):
        for line in self.proc.stdout:
            self.lines.append((time.perf_counter(), line.strip()))

    def stop(self, t0: float, t1: float) -> dict:
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        time.sleep(0.15)
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
        rows = [l for (t, l) in self.lines if t0 <= t <= t1 + 0.2] or [l for (_, l) in self.lines]
        sm, smax, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for l in rows:
            f = [x.strip() for x in l.split(",")]
            if len(f) < 9:
                continue
            try:
                sm.append(float(f[1]))
                smax.append(float(f[2]))
            except ValueError:
                continue
            for name, val in zip(names, f[5:9]):
                if val.lower().startswith("active"):
                    reasons.add(name)
        return {"sm_mhz": float(np.median(sm)) if sm else None, "sm_max_mhz": max(smax) if smax else None,
                "reasons": sorted(reasons), "samples": len(sm)}


def cpu_matvec_rate(weights, m_x, threads: int, budget_s: float):
    """Times the oracle's q4 matvec (f16 scales) on the host over `weights`, a list of distinct (scales, packed)
    matrices visited in turn (four of them are 132 MB, more than the host's caches): returns (TB/s, reps, seconds)."""
    import oracle

    oracle.build()
    x = m_x.astype(np.float64)
    for sc, pk in weights:
        oracle.qmatmul(oracle.KIND_Q4_F16, sc, pk, N_OUT, K_IN, x, threads)  # warm
    reps, t0 = 0, time.perf_counter()
    while True:
        sc, pk = weights[reps % len(weights)]
        oracle.qmatmul(oracle.KIND_Q4_F16, sc, pk, N_OUT, K_IN, x, threads)
        reps += 1
        dt = time.perf_counter() - t0
        if dt >= budget_s:
            break
    return algorithmic_bytes(x.shape[0]) * reps / dt / 1e12, reps, dt


def host_weight(seed: int):
    rng = np.random.default_rng(seed)
    packed = rng.integers(0, 256, (N_OUT, K_IN // 2), dtype=np.uint8)
    scales = rng.uniform(0.002, 0.02, (N_OUT, K_IN // GROUP)).astype(np.float16).view(np.uint16)
    return scales, packed


def run_reference(args, rank: int) -> None:
    """The reference's CPU implementation of the path (its restatement in oracle/, since the Rust
    crate cannot be built here) on all host threads.  One step = --ref-sample matvecs."""
    if rank != 0:
        return
    import oracle

    oracle.build()
    threads = oracle.max_threads()
    per_step = args.ref_sample
    weights = [host_weight(43 + i) for i in range(per_step)]      # distinct matrices: the step streams them, as the GPU arm does
    rng = np.random.default_rng(44)
    x = rng.standard_normal((args.m, K_IN)).astype(np.float32).astype(np.float64)
    for _ in range(max(args.warmup, 1)):
        for sc, pk in weights:
            oracle.qmatmul(oracle.KIND_Q4_F16, sc, pk, N_OUT, K_IN, x, threads)
    t0 = time.perf_counter()
    for _ in range(args.steps):
        for sc, pk in weights:
            oracle.qmatmul(oracle.KIND_Q4_F16, sc, pk, N_OUT, K_IN, x, threads)
    dt = time.perf_counter() - t0
    value = algorithmic_bytes(args.m) * args.steps * per_step / dt / 1e12
    sample = (f"each timed step = {per_step} distinct matrices ({per_step * algorithmic_bytes(args.m) / 1e6:.0f} MB) of the "
              f"{args.layers} a full step streams, M={args.m}, {threads} threads; the reference itself is single-threaded")
    print(json.dumps({
        "impl": "reference", "metric": METRIC, "value": value, "unit": UNIT, "n_gpus": args.gpus, "steps": args.steps,
        "warmup": args.warmup, "ms_per_step": dt / args.steps * 1e3, "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "f64", "data": "synthetic",
        "config": workload_config(args),
        "cpu_baseline": {"value": value, "unit": UNIT, "cores": threads, "kind": "port", "sample": sample},
        "e2e": {"value": value, "unit": UNIT, "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
    }))


def workload_config(args) -> dict:
    return {"workload": f"int4-g32/f16-scale dequant-GEMV K={K_IN} N={N_OUT} M={args.m} (the headline int4 GEMM configuration)",
            "layers_per_step": args.layers, "m": args.m,
            "l2": f"{args.layers} distinct weight matrices per step ({args.layers * algorithmic_bytes(args.m) / 1e6:.0f} MB) >> 126 MB L2",
            "parallelism": f"replicated column shards x{args.gpus}, no data-path collective"}


def run_ours(args, rank: int, world: int, local_rank: int) -> None:
    import torch

    import tang_b200 as tb

    torch.cuda.set_device(local_rank)
    if world > 1:
        import torch.distributed as dist

        dist.init_process_group("nccl", device_id=torch.device("cuda", local_rank))
    # The context owns its stream (on a stream of its own the library may let independent matvecs overlap);
    # torch sees the same stream, so CUDA events recorded through torch time the library's launches.
    dev = tb.QuantComputeDevice(local_rank)
    stream = torch.cuda.ExternalStream(dev.stream, device=torch.device("cuda", local_rank))
    L, m = args.layers, args.m

    with torch.cuda.stream(stream):
        gen = torch.Generator(device="cuda").manual_seed(43 + rank)
        packed = torch.randint(0, 256, (L, N_OUT, K_IN // 2), dtype=torch.uint8, device="cuda", generator=gen)
        scales = (torch.rand((L, N_OUT, K_IN // GROUP), device="cuda", generator=gen) * 0.018 + 0.002).half()
        x = torch.randn((m, K_IN), device="cuda", generator=gen).bfloat16()
        y = torch.empty((L, m, N_OUT), dtype=torch.bfloat16, device="cuda")
    stream.synchronize()
    L_ = dev._L
    import ctypes as C

    handles = []
    for i in range(L):
        h = C.c_void_p()
        dev._check(L_.tq_qweight_from_device_arrays(dev._ctx, tb.Q4_F16, C.c_void_p(packed[i].data_ptr()),
                                             C.c_void_p(scales[i].data_ptr()), N_OUT, K_IN, C.byref(h)))
        handles.append(h)

    def one_pass():
        for i in range(L):
            dev._check(L_.tq_qlinear(dev._ctx, handles[i], C.c_void_p(x.data_ptr()), tb.BF16, 0, m,
                                     C.c_void_p(y[i].data_ptr()), tb.BF16, 0, None))

    one_pass()          # eager once: sizes workspaces, sets kernel attributes
    dev.sync()
    dev.begin_capture()
    one_pass()
    graph = dev.end_capture()

    # parity spot check against the oracle on rank 0 (256 output rows of layer 0)
    parity = None
    if rank == 0:
        import oracle

        oracle.build()
        rows = 256
        sc_h = scales[0, :rows].cpu().numpy().view(np.uint16)
        pk_h = packed[0, :rows].cpu().numpy()
        x_h = x.float().cpu().numpy().astype(np.float64)
        want = oracle.qmatmul(oracle.KIND_Q4_F16, sc_h, pk_h, rows, K_IN, x_h, 0)
        got = y[0, :, :rows].float().cpu().numpy().astype(np.float64)
        rms = float(np.sqrt(np.mean(want * want)))
        parity = float(np.max(np.abs(got - want) / np.maximum(np.abs(want), 1e-2 * rms)))

    def barrier():
        if world > 1:
            import torch.distributed as dist

            dist.barrier()
        torch.cuda.synchronize()

    sampler = ClockSampler(local_rank) if rank == 0 else None
    if sampler:
        sampler.start()
    for _ in range(args.warmup):
        graph.launch()
    barrier()
    launches0 = dev.launch_count
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    t_wall0 = time.perf_counter()
    with torch.cuda.stream(stream):
        ev0.record(stream)
        for _ in range(args.steps):
            graph.launch()
        ev1.record(stream)
    barrier()
    t_wall1 = time.perf_counter()
    ms = ev0.elapsed_time(ev1)
    gpu_launches = dev.launch_count - launches0

    # ---- end to end: the reference-shaped host call, pinned host vectors, copies inside the timing.  A step queues
    # the L matvecs (upload of x, kernel, result written to its own pinned vector) and waits once for all of them;
    # the second timing waits after every call, as a loop over the reference's q4_matvec does.
    # Every matrix of the step gets its own pinned input vector (a layer's input differs from the next one's).
    xh = torch.empty((L, m, K_IN), dtype=torch.bfloat16).pin_memory()
    xh.copy_(torch.randn((L, m, K_IN), generator=torch.Generator().manual_seed(7 + rank)).bfloat16())
    yh = torch.empty((L, m, N_OUT), dtype=torch.bfloat16).pin_memory()

    x_ptrs = [C.c_void_p(xh[i].data_ptr()) for i in range(L)]      # (a caller has its pointers at hand)
    y_ptrs = [C.c_void_p(yh[i].data_ptr()) for i in range(L)]

    def e2e_pass(call):
        for i in range(L):
            dev._check(call(dev._ctx, handles[i], x_ptrs[i], y_ptrs[i], tb.BF16, m))

    # Timed on the host clock, from the first call to the return of the last wait (the clock an end-to-end caller
    # sees); the CUDA-event time of the same region is kept beside it.
    e2e_steps = max(1, min(args.steps, 20))
    e2e_times, e2e_event_times = [], []
    for call, wait in ((L_.tq_q_matvec_host, False), (L_.tq_q_matvec_host_async, True)):
        e2e_pass(call)
        dev.sync()
        barrier()
        with torch.cuda.stream(stream):
            ev0.record(stream)
            t0 = time.perf_counter()
            for _ in range(e2e_steps):
                e2e_pass(call)
                if wait:
                    dev.sync()          # the step's results are read here: one wait per step
            t1 = time.perf_counter()
            ev1.record(stream)
        barrier()
        e2e_times.append((t1 - t0) * 1e3)
        e2e_event_times.append(ev0.elapsed_time(ev1))
    e2e_sync_ms, e2e_async_ms = e2e_times
    # The same step recorded once (tq_graph_begin .. tq_graph_end around the L calls) and replayed: every replay reads
    # the pinned input vectors again and writes the pinned results; per step the host launches one graph and waits once.
    yh_calls = yh.clone()                    # what the call-by-call loop above produced
    dev.begin_capture()
    e2e_pass(L_.tq_q_matvec_host_async)
    e2e_graph = dev.end_capture()
    yh.zero_()
    e2e_graph.launch()
    dev.sync()
    e2e_graph_ok = bool(torch.equal(yh.view(torch.int16), yh_calls.view(torch.int16)))
    barrier()
    with torch.cuda.stream(stream):
        ev0.record(stream)
        t0 = time.perf_counter()
        for _ in range(e2e_steps):
            e2e_graph.launch()
            dev.sync()
        t1 = time.perf_counter()
        ev1.record(stream)
    barrier()
    e2e_ms = (t1 - t0) * 1e3
    e2e_event_times.append(ev0.elapsed_time(ev1))
    e2e_graph.free()
    clocks = sampler.stop(t_wall0, t_wall1) if sampler else None

    t = torch.tensor([ms, e2e_ms, e2e_sync_ms, e2e_async_ms], dtype=torch.float64, device="cuda")
    if world > 1:
        import torch.distributed as dist

        dist.all_reduce(t, op=dist.ReduceOp.MAX)
    ms, e2e_ms, e2e_sync_ms, e2e_async_ms = float(t[0]), float(t[1]), float(t[2]), float(t[3])

    host_w = None   # layer 0 on the host, for the CPU baseline leg
    if rank == 0 and world == 1 and not args.no_cpu_baseline:
        host_w = (scales[0].cpu().numpy().view(np.uint16), packed[0].cpu().numpy(), x.float().cpu().numpy())

    # ---- Llama-3-8B-shaped decode step, tensor parallel over the ranks of this job
    decode = None
    comm = None
    if world > 1 and not (args.no_decode and args.no_extras):
        import torch.distributed as dist

        ids = [tb.Comm.unique_id() if rank == 0 else None]
        dist.broadcast_object_list(ids, src=0)
        comm = tb.Comm(dev, ids[0], rank, world)
        comm.enable_peer(64 * 7168)      # the row-parallel sums of a decode step (<= 64 rows of d_model f32) go over peer memory
    if not args.no_decode:
        graph.free()
        graph = None
        for h in handles:
            L_.tq_qweight_free(dev._ctx, h)
        del packed, scales, y
        torch.cuda.empty_cache()
        decode = run_decode(dev, tb, torch, stream, comm, rank, world, args, barrier)

    extras = None
    if not args.no_extras:
        if graph is not None:
            graph.free()
            graph = None
        torch.cuda.empty_cache()
        peak_gbs = measured_peaks()[0]
        extras = run_extras(dev, tb, torch, stream, peak_gbs) if world == 1 else {}
        extras.update(run_sharded_extras(dev, tb, torch, stream, peak_gbs, comm, rank, world, barrier))
    if comm:
        comm.destroy()

    if rank == 0:
        bytes_launch = algorithmic_bytes(m)
        ms_per_step = ms / args.steps
        value = world * L * bytes_launch / (ms_per_step * 1e-3) / 1e12
        e2e_value = world * L * bytes_launch / (e2e_ms / e2e_steps * 1e-3) / 1e12
        peak, peak_kind = measured_peaks()
        achieved = bytes_launch / (ms_per_step * 1e-3 / L) / 1e9
        cpu = None
        if world == 1 and not args.no_cpu_baseline:
            import oracle

            threads = oracle.max_threads()
            weights = [(host_w[0], host_w[1])] + [host_weight(900 + i) for i in range(3)]
            v, reps, dt = cpu_matvec_rate(weights, host_w[2], threads, args.cpu_budget)
            # the reference runs this loop on one thread (README: "single-threaded"): that figure beside the all-core one
            v1, reps1, dt1 = cpu_matvec_rate(weights, host_w[2], 1, args.cpu_budget)
            cpu = {"value": v, "unit": UNIT, "cores": threads, "kind": "port",
                   "sample": f"{reps} matvecs over 4 distinct K={K_IN} N={N_OUT} matrices, M={m}, in {dt:.1f} s",
                   "single_thread": {"value": v1, "unit": UNIT, "cores": 1,
                                     "sample": f"{reps1} matvecs over the same 4 matrices in {dt1:.1f} s"}}
        out = {
            "metric": METRIC, "value": value, "unit": UNIT, "n_gpus": world, "steps": args.steps, "warmup": args.warmup,
            "ms_per_step": ms_per_step, "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
            "dtype": "int4 weights x bf16 activations, f32 accumulate", "data": "synthetic",
            "config": workload_config(args),
            "pct_of_8tbps_nominal": 100.0 * value / world / 8.0,
            "roofline": {"bound": "hbm", "achieved": achieved, "peak": peak, "unit": "GB/s", "frac": achieved / peak,
                         "peak_source": peak_kind, "traffic": NCU_TRAFFIC_BYTES_PER_LAUNCH,
                         "kernel": "qgemv_sk_kernel<Q4_F16> (persistent GEMV)" if m == 1 else "qgemm_sk_kernel (2..8 rows) / qgemm_mma_kernel / qgemm_umma_kernel", "algorithmic_bytes_per_launch": bytes_launch,
                         "avg_launch_us": ms_per_step * 1e3 / L},
            "e2e": {"value": e2e_value, "unit": UNIT, "h2d_bytes_per_step": L * m * K_IN * 2,
                    "d2h_bytes_per_step": L * m * N_OUT * 2, "steps": e2e_steps,
                    "call": "tq_graph_launch of a recorded step (L x tq_q_matvec_host_async: pinned host vectors, one per matrix, read "
                            "again by every replay; results written to pinned host vectors) + one tq_sync per step",
                    "clock": "host wall clock around the calls and their final wait",
                    "graph_result_equals_call_by_call": e2e_graph_ok,
                    "value_cuda_events": world * L * bytes_launch / (e2e_event_times[2] / e2e_steps * 1e-3) / 1e12,
                    "value_async_calls": world * L * bytes_launch / (e2e_async_ms / e2e_steps * 1e-3) / 1e12,
                    "call_async_calls": "tq_q_matvec_host_async per matrix + one tq_sync per step, no graph",
                    "value_wait_per_call": world * L * bytes_launch / (e2e_sync_ms / e2e_steps * 1e-3) / 1e12,
                    "call_wait_per_call": "tq_q_matvec_host (q4_matvec: returns when the result is on the host)"},
            "cpu_baseline": cpu, "gpu_launches": int(gpu_launches), "clocks": clocks,
            "parity_max_rel_err_vs_oracle": parity,
            "decode": None if decode is None else {
                "metric": "llama3_8b_shape_decode_tokens_per_s", "peak_gbs": peak,
                "results": [dict(r, frac_of_hbm_peak=r["gbs_per_gpu"] / peak) for r in decode if "batch" in r],
                "prefill": [r for r in decode if "prefill_tokens" in r]},
            "extras": extras,
        }
        print(json.dumps(out))
    if graph is not None:
        graph.free()
    if world > 1:
        import torch.distributed as dist

        dist.destroy_process_group()


# ----------------------------------------------------------------------------------------------
# Llama-3-8B-shaped decode step (the decode configuration): 32 layers, d 4096, 32/8 heads of 128, FFN
# 14336, vocab 128256, int4-g32/f16 weights, bf16 KV cache prefilled to 2048 positions; tensor
# parallel over the ranks of this job.  Random-init weights generated on the device.
# ----------------------------------------------------------------------------------------------
LLAMA = dict(n_layers=32, d=4096, n_heads=32, n_kv=8, hd=128, ffn=14336, vocab=128256, ctx=2048)


def decode_bytes_per_gpu(batch: int, tp: int, n_layers: int) -> int:
    """Algorithmic bytes one GPU streams per step: its weight shards (nibbles + f16 scales) + its KV heads."""
    c = LLAMA
    per_layer_w = (c["d"] * (c["n_heads"] + 2 * c["n_kv"]) * c["hd"] + c["d"] * c["n_heads"] * c["hd"] + 3 * c["d"] * c["ffn"])
    w = n_layers * per_layer_w + c["vocab"] * c["d"]
    wbytes = w // 2 + w // 32 * 2
    kv = n_layers * 2 * batch * (c["ctx"] + 1) * c["n_kv"] * c["hd"] * 2
    return (wbytes + kv) // tp


def build_llama(dev, tb, torch, stream, comm, rank, world, n_layers, max_batch, c=None):
    import ctypes as C

    c = c or LLAMA
    tp = world
    hl, kl, fl, vl = c["n_heads"] // tp, c["n_kv"] // tp, c["ffn"] // tp, c["vocab"] // tp
    d, hd = c["d"], c["hd"]
    cfg = tb.LlamaConfig(n_layers, d, c["n_heads"], c["n_kv"], hd, c["ffn"], c["vocab"], c["ctx"] + 1, max_batch, 1e-5, 500000.0)
    model = tb.LlamaModel(dev, cfg, comm)
    gen = torch.Generator(device="cuda").manual_seed(1000 + rank)
    keep = []

    def qw(rows, cols):
        with torch.cuda.stream(stream):
            pay = torch.randint(0, 256, (rows, cols // 2), dtype=torch.uint8, device="cuda", generator=gen)
            sc = (torch.rand((rows, cols // 32), device="cuda", generator=gen) * 0.018 + 0.002).half()
        stream.synchronize()
        w = dev.qweight_from_device(tb.Q4_F16, pay.data_ptr(), sc.data_ptr(), rows, cols)
        dev.sync()
        return w

    def bf16_vec(n, std=0.02):
        with torch.cuda.stream(stream):
            t = (torch.randn(n, device="cuda", generator=gen) * std).bfloat16()
        stream.synchronize()
        keep.append(t)
        return tb.Buffer(dev, t.data_ptr(), t.numel(), tb.BF16, owns=False)

    for l in range(n_layers):
        # gate/up in the interleaved row order: the SwiGLU becomes the projection's epilogue
        model.set_layer(l, tb.LlamaLayerWeights(qw((hl + 2 * kl) * hd, d), qw(d, hl * hd), dev.interleave_gate_up(qw(2 * fl, d)), qw(d, fl),
                                                bf16_vec(d), bf16_vec(d)))
        kbuf, vbuf, _ = model.kv_buffers(l)
        with torch.cuda.stream(stream):     # prefill the cache with bf16 N(0,1), in slices to bound the temporary
            step = 1 << 26
            for buf in (kbuf, vbuf):
                for off in range(0, buf.n, step):
                    n = min(step, buf.n - off)
                    t = torch.randn(n, device="cuda", generator=gen).bfloat16()
                    dev._check(dev._L.tq_convert(dev._ctx, C.c_void_p(t.data_ptr()), tb.BF16, C.c_void_p(buf.ptr + 2 * off), tb.BF16, n))
                    stream.synchronize()
    model.set_head(bf16_vec(c["vocab"] * d), bf16_vec(d), qw(vl, d))
    model._bench_keep = keep
    return model


def run_decode(dev, tb, torch, stream, comm, rank, world, args, barrier):
    """Times the decode step at each batch size; returns a list of result dicts (rank 0 uses them)."""
    c = LLAMA
    batches = [int(b) for b in args.decode_batches.split(",") if b]
    model = build_llama(dev, tb, torch, stream, comm, rank, world, args.decode_layers, max(batches))
    out = []
    for B in batches:
        with torch.cuda.stream(stream):
            tok = torch.randint(0, c["vocab"], (B,), dtype=torch.int32, device="cuda")
            pos = torch.full((B,), c["ctx"], dtype=torch.int32, device="cuda")
            logits = torch.empty((world, B, c["vocab"] // world), dtype=torch.float32, device="cuda")
        stream.synchronize()
        tbuf = tb.Buffer(dev, tok.data_ptr(), B, tb.I32, owns=False)
        pbuf = tb.Buffer(dev, pos.data_ptr(), B, tb.I32, owns=False)
        lbuf = tb.Buffer(dev, logits.data_ptr(), logits.numel(), tb.F32, owns=False)
        model.decode(tbuf, pbuf, B, c["ctx"] + 1, lbuf)      # eager once (workspaces, attributes, NCCL warm-up)
        dev.sync()
        l0 = dev.launch_count
        dev.begin_capture()
        model.decode(tbuf, pbuf, B, c["ctx"] + 1, lbuf)
        graph = dev.end_capture()
        for _ in range(max(args.warmup, 3)):
            graph.launch()
        barrier()
        ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        steps = args.decode_steps
        with torch.cuda.stream(stream):
            ev0.record(stream)
            for _ in range(steps):
                graph.launch()
            ev1.record(stream)
        barrier()
        ms = ev0.elapsed_time(ev1) / steps
        t = torch.tensor([ms], dtype=torch.float64, device="cuda")
        if world > 1:
            import torch.distributed as dist

            dist.all_reduce(t, op=dist.ReduceOp.MAX)
        ms = float(t[0])
        finite = bool(torch.isfinite(logits).all().item())
        graph.free()
        byt = decode_bytes_per_gpu(B, world, args.decode_layers)
        out.append({"batch": B, "tp": world, "layers": args.decode_layers, "ms_per_step": ms, "tokens_per_s": B / (ms * 1e-3),
                    "bytes_per_gpu": byt, "gbs_per_gpu": byt / (ms * 1e-3) / 1e9, "logits_finite": finite,
                    "kernels_per_step": int((dev.launch_count - l0) // (steps + max(args.warmup, 3)))})
    # prompt processing with the same model: one sequence, a 2048-token chunk from an empty cache
    q_len = min(2048, c["ctx"])
    with torch.cuda.stream(stream):
        ptok = torch.randint(0, c["vocab"], (q_len,), dtype=torch.int32, device="cuda")
        start0 = torch.zeros((1,), dtype=torch.int32, device="cuda")
        plog = torch.empty((world, 1, c["vocab"] // world), dtype=torch.float32, device="cuda")
    stream.synchronize()
    mk = lambda t, dt: tb.Buffer(dev, t.data_ptr(), t.numel(), dt, owns=False)
    model.prefill(mk(ptok, tb.I32), mk(start0, tb.I32), 1, q_len, mk(plog, tb.F32))      # sizes the workspaces
    dev.sync()
    barrier()
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    reps = 3
    with torch.cuda.stream(stream):
        ev0.record(stream)
        for _ in range(reps):
            model.prefill(mk(ptok, tb.I32), mk(start0, tb.I32), 1, q_len, mk(plog, tb.F32))
        ev1.record(stream)
    barrier()
    pms = ev0.elapsed_time(ev1) / reps
    t = torch.tensor([pms], dtype=torch.float64, device="cuda")
    if world > 1:
        import torch.distributed as dist

        dist.all_reduce(t, op=dist.ReduceOp.MAX)
    pms = float(t[0])
    w_params = args.decode_layers * (c["d"] * (c["n_heads"] + 2 * c["n_kv"]) * c["hd"] + c["d"] * c["n_heads"] * c["hd"] + 3 * c["d"] * c["ffn"])
    out.append({"prefill_tokens": q_len, "tp": world, "layers": args.decode_layers, "ms": pms, "tokens_per_s": q_len / (pms * 1e-3),
                "tflops_per_gpu": 2.0 * q_len * w_params / world / (pms * 1e-3) / 1e12, "logits_finite": bool(torch.isfinite(plog).all().item())})
    model.destroy()
    return out


# ----------------------------------------------------------------------------------------------
# The other benchmark configurations, timed briefly at N=1 and reported under "extras": the M sweep of
# the int4 GEMM, the DeepSeek-V2-Lite-shaped MoE layer and the DeepSeek-V3-shaped MLA decode
# attention.  Seeded synthetic inputs generated on the device.
# ----------------------------------------------------------------------------------------------
def _time_ms(torch, stream, dev, fn, reps, warm=2):
    for _ in range(warm):
        fn()
    dev.sync()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    with torch.cuda.stream(stream):
        e0.record(stream)
        for _ in range(reps):
            fn()
        e1.record(stream)
    dev.sync()
    return e0.elapsed_time(e1) / reps


def run_extras(dev, tb, torch, stream, peak_gbs):
    import ctypes as C

    L_ = dev._L
    gen = torch.Generator(device="cuda").manual_seed(77)
    out = {}

    def q4(rows, cols):
        with torch.cuda.stream(stream):
            pay = torch.randint(0, 256, (rows, cols // 2), dtype=torch.uint8, device="cuda", generator=gen)
            sc = (torch.rand((rows, cols // 32), device="cuda", generator=gen) * 0.018 + 0.002).half()
        stream.synchronize()
        w = dev.qweight_from_device(tb.Q4_F16, pay.data_ptr(), sc.data_ptr(), rows, cols)
        dev.sync()
        return w

    def i8(rows, cols):
        with torch.cuda.stream(stream):
            pay = torch.randint(-127, 128, (rows, cols), dtype=torch.int8, device="cuda", generator=gen)
            sc = torch.rand(rows, device="cuda", generator=gen) * 0.009 + 0.001
        stream.synchronize()
        w = dev.qweight_from_device(tb.I8_ROW, pay.data_ptr(), sc.data_ptr(), rows, cols)
        dev.sync()
        return w

    def bf16(shape, std=1.0):
        with torch.cuda.stream(stream):
            t = (torch.randn(shape, device="cuda", generator=gen) * std).bfloat16()
        stream.synchronize()
        return t

    # ---- the int8 GEMV of the CPU-runnable configuration: [4096, 4096] int8, one f32 scale per output row (and the same
    # integers as tang-infer's native Q8 blocks, one f32 scale per 32 weights), f32 activations, f32 results;
    # 16 distinct matrices per graph (268 MB > L2)
    def q8_blocks(rows, cols):
        with torch.cuda.stream(stream):
            pay = torch.randint(-127, 128, (rows, cols), dtype=torch.int8, device="cuda", generator=gen)
            sc = (torch.rand((rows, cols // 32), device="cuda", generator=gen) * 0.009 + 0.001)
        stream.synchronize()
        w = dev.qweight_from_device(tb.Q8_F32, pay.data_ptr(), sc.data_ptr(), rows, cols)
        dev.sync()
        return w

    int8 = []
    n8 = 16
    for name, make, byt in (("int8 per-row scale", i8, 4096 * 4096 + 4096 * 4 + 4096 * 4 + 4096 * 4),
                            ("Q8 blocks (f32 scale per 32)", q8_blocks, 4096 * 4096 + 4096 * 128 * 4 + 4096 * 4 + 4096 * 4)):
        w8 = [make(4096, 4096) for _ in range(n8)]
        with torch.cuda.stream(stream):
            x32 = torch.randn((1, 4096), device="cuda", generator=gen)
        xb16 = x32.bfloat16()
        y32 = torch.empty((n8, 1, 4096), dtype=torch.float32, device="cuda")
        stream.synchronize()
        row = {"layout": name, "algorithmic_bytes": byt}
        for tag, xt, xdt in (("f32_x", x32, tb.F32), ("bf16_x", xb16, tb.BF16)):
            def one8():
                for i, w in enumerate(w8):
                    dev._check(L_.tq_qlinear(dev._ctx, C.c_void_p(w.handle), C.c_void_p(xt.data_ptr()), xdt, 0, 1,
                                             C.c_void_p(y32[i].data_ptr()), tb.F32, 0, None))
            one8()
            dev.sync()
            dev.begin_capture()
            one8()
            g = dev.end_capture()
            us = _time_ms(torch, stream, dev, g.launch, 10, 3) * 1e3 / n8
            g.free()
            row[tag] = {"us_per_launch": us, "gbs": byt / us / 1e3, "frac_of_hbm_peak": byt / us / 1e3 / peak_gbs}
        # the same weights against many rows (the tcgen05 GEMM): bf16 activations, f32 results
        for m in (64, 2048):
            xm = bf16((m, 4096))
            ym = torch.empty((n8, m, 4096), dtype=torch.float32, device="cuda")
            stream.synchronize()

            def many8():
                for i, w in enumerate(w8):
                    dev._check(L_.tq_qlinear(dev._ctx, C.c_void_p(w.handle), C.c_void_p(xm.data_ptr()), tb.BF16, 0, m,
                                             C.c_void_p(ym[i].data_ptr()), tb.F32, 0, None))
            many8()
            dev.sync()
            dev.begin_capture()
            many8()
            g = dev.end_capture()
            us = _time_ms(torch, stream, dev, g.launch, 10, 3) * 1e3 / n8
            g.free()
            row["m%d_bf16_x" % m] = {"us_per_launch": us, "tflops": 2.0 * m * 4096 * 4096 / us / 1e6}
            del xm, ym
        int8.append(row)
        for w in w8:
            w.free()
    out["int8_gemv_4096"] = int8

    # ---- the reference's one published number for this path: quantize/q8_matvec_576x576, 207 992 ns on an Apple M4 Max,
    # one thread (crates/tang-bench/benches/cpu_training.rs:267-275).  Here: the oracle port on one host thread, the
    # reference-shaped host call (f64 vectors in and out, waits), and the kernel alone from a graph.
    import oracle

    oracle.build()
    rng = np.random.default_rng(576)
    wf = (rng.standard_normal((576, 576)) * 0.05).astype(np.float32)
    s8, v8 = oracle.quantize_matrix_q8(wf, 576, 576)
    xq = rng.standard_normal(576)
    t0 = time.perf_counter()
    n_cpu = 200
    for _ in range(n_cpu):
        oracle.q8_matvec(s8, v8, 576, 576, xq, 1)
    cpu_ns = (time.perf_counter() - t0) / n_cpu * 1e9
    w576 = dev.upload_q8(tb.QuantizedQ8(s8.reshape(-1), v8.reshape(-1), (576, 576)))
    dev.q8_matvec(w576, xq)
    t0 = time.perf_counter()
    for _ in range(200):
        dev.q8_matvec(w576, xq)
    host_call_ns = (time.perf_counter() - t0) / 200 * 1e9
    with torch.cuda.stream(stream):
        x576 = torch.randn((1, 576), device="cuda", generator=gen)
    y576 = torch.empty((1, 576), dtype=torch.float32, device="cuda")
    stream.synchronize()

    def one576():
        dev._check(L_.tq_qlinear(dev._ctx, C.c_void_p(w576.handle), C.c_void_p(x576.data_ptr()), tb.F32, 0, 1,
                                 C.c_void_p(y576.data_ptr()), tb.F32, 0, None))
    one576()
    dev.sync()
    dev.begin_capture()
    for _ in range(20):
        one576()
    g = dev.end_capture()
    kern_ns = _time_ms(torch, stream, dev, g.launch, 10, 3) * 1e6 / 20
    g.free()
    out["q8_matvec_576x576"] = {"reference_published_ns_m4max_1thread": 207992, "oracle_port_1thread_ns": cpu_ns,
                                "host_call_f64_ns": host_call_ns, "device_launches_from_graph_ns": kern_ns}

    # ---- int4 GEMM: M sweep over 16 distinct matrices (528 MB > L2), bf16 results, one CUDA graph per M
    n_mat = 16
    ws = [q4(N_OUT, K_IN) for _ in range(n_mat)]
    sweep = []
    for m in (1, 8, 32, 64, 512, 2048):
        x = bf16((m, K_IN))
        y = torch.empty((n_mat, m, N_OUT), dtype=torch.bfloat16, device="cuda")   # one result per matrix, as in the headline

        def one():
            for i, w in enumerate(ws):
                dev._check(L_.tq_qlinear(dev._ctx, C.c_void_p(w.handle), C.c_void_p(x.data_ptr()), tb.BF16, 0, m,
                                         C.c_void_p(y[i].data_ptr()), tb.BF16, 0, None))
        one()
        dev.sync()
        dev.begin_capture()
        one()
        g = dev.end_capture()
        us = _time_ms(torch, stream, dev, g.launch, 10, 3) * 1e3 / n_mat
        g.free()
        byt, fl = algorithmic_bytes(m), 2.0 * m * N_OUT * K_IN
        sweep.append({"m": m, "us_per_launch": us, "gbs": byt / us / 1e3, "tflops": fl / us / 1e6,
                      "frac_of_hbm_peak": byt / us / 1e3 / peak_gbs})
    out["int4_gemm_m_sweep"] = sweep
    for w in ws:
        w.free()
    del ws
    torch.cuda.empty_cache()

    # ---- prefill attention: one sequence, Llama-3-8B heads (32 query / 8 KV heads of 128), causal chunk of q_len positions
    pre = []
    for q_len in (512, 2048):
        nh, nkv, hd = 32, 8, 128
        q = bf16((1, q_len, nh * hd))
        kc, vc = bf16((1, q_len, nkv * hd)), bf16((1, q_len, nkv * hd))
        o = torch.empty((1, q_len, nh * hd), dtype=torch.bfloat16, device="cuda")
        st0 = dev.upload(np.zeros(1, np.int32), tb.I32)

        def fn():
            dev._check(L_.tq_gqa_prefill(dev._ctx, C.c_void_p(q.data_ptr()), C.c_void_p(kc.data_ptr()), C.c_void_p(vc.data_ptr()),
                                         C.c_void_p(st0.ptr), 1, q_len, nh, nkv, hd, q_len * nkv * hd, C.c_void_p(o.data_ptr()), tb.BF16))
        ms = _time_ms(torch, stream, dev, fn, 10, 3)
        flops = 4.0 * nh * hd * q_len * (q_len + 1) / 2          # QK^T and PV over the causal half
        pre.append({"q_len": q_len, "us": ms * 1e3, "tflops": flops / ms / 1e9})
    out["gqa_prefill_llama_heads"] = pre
    return out


def run_sharded_extras(dev, tb, torch, stream, peak_gbs, comm, rank, world, barrier):
    """The MoE layer with its experts over the ranks and the MLA layer with its heads over the ranks; at N = 1 the
    same calls without a communicator.  Times are the max over the ranks."""
    import ctypes as C

    L_ = dev._L
    gen = torch.Generator(device="cuda").manual_seed(77)      # same seed on every rank: replicated tensors are equal
    out = {}

    def q4(rows, cols):
        with torch.cuda.stream(stream):
            pay = torch.randint(0, 256, (rows, cols // 2), dtype=torch.uint8, device="cuda", generator=gen)
            sc = (torch.rand((rows, cols // 32), device="cuda", generator=gen) * 0.018 + 0.002).half()
        stream.synchronize()
        w = dev.qweight_from_device(tb.Q4_F16, pay.data_ptr(), sc.data_ptr(), rows, cols)
        dev.sync()
        return w

    def i8(rows, cols):
        with torch.cuda.stream(stream):
            pay = torch.randint(-127, 128, (rows, cols), dtype=torch.int8, device="cuda", generator=gen)
            sc = torch.rand(rows, device="cuda", generator=gen) * 0.009 + 0.001
        stream.synchronize()
        w = dev.qweight_from_device(tb.I8_ROW, pay.data_ptr(), sc.data_ptr(), rows, cols)
        dev.sync()
        return w

    def bf16(shape, std=1.0):
        with torch.cuda.stream(stream):
            t = (torch.randn(shape, device="cuda", generator=gen) * std).bfloat16()
        stream.synchronize()
        return t

    def timed(fn, reps):
        fn()
        dev.sync()
        dev.begin_capture()
        fn()
        g = dev.end_capture()
        barrier()
        ms = _time_ms(torch, stream, dev, g.launch, reps)
        g.free()
        if world > 1:
            import torch.distributed as dist

            t = torch.tensor([ms], dtype=torch.float64, device="cuda")
            dist.all_reduce(t, op=dist.ReduceOp.MAX)
            ms = float(t[0])
        return ms

    # ---- MoE layer, d 2048, 64 routed + 2 shared experts of width 1408, top-6; experts over the ranks
    d, ffn, E, k, nsh = 2048, 1408, 64, 6, 2
    n_local = E // world
    wg = bf16((E, d), 0.02)
    layer = tb.MoeLayer(dev, tb.MoeConfig(d, ffn, E, k, nsh, 0, rank, world), tb.Buffer(dev, wg.data_ptr(), wg.numel(), tb.BF16, owns=False),
                        q4(n_local * 2 * ffn, d), q4(n_local * d, ffn), [q4(2 * ffn, d) for _ in range(nsh)], [q4(d, ffn) for _ in range(nsh)])
    per_expert = 3 * (ffn * d // 2 + ffn * d // 32 * 2)
    moe = []
    for T in (1, 64, 256, 4096):
        h = bf16((T, d))                                      # the same tokens on every rank
        hb = tb.Buffer(dev, h.data_ptr(), h.numel(), tb.BF16, owns=False)
        o, idx, _w = layer.forward(hb, T, comm=comm, want_routing=True)
        dev.sync()
        distinct = int(len(set(idx.to_vec().tolist())))
        ob = dev.alloc(T * d, tb.F32)
        reps = 10 if T <= 256 else 3
        ms = timed(lambda: layer.forward(hb, T, out=ob, comm=comm), reps)
        byt = (distinct + nsh) * per_expert
        row = {"tokens": T, "us": ms * 1e3, "distinct_routed_experts": distinct, "weight_bytes_touched": byt,
               "gbs": byt / ms / 1e6, "tflops": 2.0 * T * (k + nsh) * 3 * ffn * d / ms / 1e9,
               "form": "one GPU" if world == 1 else "tokens replicated, experts over the ranks, all-reduce of the outputs"}
        if world > 1 and T % world == 0:
            # tokens sharded over the ranks: all-to-all dispatch to the experts' owners and all-to-all combine back
            tl = T // world
            hl = tb.Buffer(dev, h[rank * tl:(rank + 1) * tl].data_ptr(), tl * d, tb.BF16, owns=False)
            ol = dev.alloc(tl * d, tb.F32)
            ms2 = timed(lambda: layer.forward_dispatch(hl, tl, comm=comm, out=ol), reps)
            row["dispatch"] = {"us": ms2 * 1e3, "tokens_per_rank": tl, "tflops": 2.0 * T * (k + nsh) * 3 * ffn * d / ms2 / 1e9,
                               "form": "tokens over the ranks, all-to-all dispatch and combine, peer blocks padded to the worst case "
                                       "(fixed size: replayed from a graph)"}
            if tl * k >= 256:
                # outside a graph the call exchanges the row counts first and sends true sizes (one host round trip inside)
                barrier()
                ms3 = _time_ms(torch, stream, dev, lambda: layer.forward_dispatch(hl, tl, comm=comm, out=ol), reps)
                if world > 1:
                    import torch.distributed as dist

                    t3 = torch.tensor([ms3], dtype=torch.float64, device="cuda")
                    dist.all_reduce(t3, op=dist.ReduceOp.MAX)
                    ms3 = float(t3[0])
                row["dispatch_counts_first"] = {"us": ms3 * 1e3, "tflops": 2.0 * T * (k + nsh) * 3 * ffn * d / ms3 / 1e9,
                                                "form": "the same call made eagerly: counts exchanged first, rows sent with their true sizes"}
        moe.append(row)
    out["moe_dsv2_lite_layer"] = moe
    layer.destroy()
    torch.cuda.empty_cache()

    # ---- MLA decode, 128 heads over the ranks, latent 512 + rope 64, int8 per-row weights.  The attention core
    # (absorb W_UK, attend over the latent cache, un-absorb W_UV) and the whole layer with q_a [1536, d], q_b and the
    # row-parallel W_O at d_model 7168 (an assumption: the configuration names no hidden size).
    H, NOPE, VD, CL, RP, QL, DM = 128 // world, 128, 128, 512, 64, 1536, 7168
    wq, wu = i8(H * CL, NOPE), i8(H * VD, CL)
    max_pos = 32768 + 1
    gain = bf16((QL,), 0.03)
    mlayer = tb.MlaLayer(dev, tb.MlaConfig(DM, H, QL, CL, NOPE, RP, VD, 64, max_pos, 1e-6), i8(QL, DM),
                         tb.Buffer(dev, gain.data_ptr(), QL, tb.BF16, owns=False), i8(H * (NOPE + RP), QL), wq, wu, i8(DM, H * VD))
    mla = []
    for ctx, B in ((4096, 1), (16384, 16), (32768, 64)):
        cache = torch.empty((B, ctx, CL + RP), dtype=torch.bfloat16, device="cuda")
        with torch.cuda.stream(stream):
            for b in range(B):
                cache[b].copy_(torch.randn((ctx, CL + RP), device="cuda", generator=gen))
        stream.synchronize()
        qn, qr = bf16((B, H, NOPE)), bf16((B, H, RP))
        hid = bf16((B, DM))
        lens = dev.upload(np.full(B, ctx, np.int32), tb.I32)
        q_full, o_lat, o = dev.alloc(B * H * (CL + RP), tb.BF16), dev.alloc(B * H * CL, tb.BF16), dev.alloc(B * H * VD, tb.F32)
        lo = dev.alloc(B * DM, tb.F32)
        cb = tb.Buffer(dev, cache.data_ptr(), cache.numel(), tb.BF16, owns=False)
        hb = tb.Buffer(dev, hid.data_ptr(), hid.numel(), tb.BF16, owns=False)

        def core():   # absorb W_UK into q, attend over the latent cache, un-absorb with W_UV
            dev._check(L_.tq_mla_absorb_q(dev._ctx, C.c_void_p(wq.handle), C.c_void_p(qn.data_ptr()), C.c_void_p(qr.data_ptr()),
                                          B, H, NOPE, C.c_void_p(q_full.ptr)))
            dev._check(L_.tq_mla_decode(dev._ctx, C.c_void_p(q_full.ptr), C.c_void_p(cache.data_ptr()), C.c_void_p(lens.ptr), B, H,
                                        CL, RP, ctx * (CL + RP), ctx, 1.0 / (NOPE + RP) ** 0.5, C.c_void_p(o_lat.ptr)))
            dev._check(L_.tq_mla_unabsorb(dev._ctx, C.c_void_p(wu.handle), C.c_void_p(o_lat.ptr), B, H, VD, C.c_void_p(o.ptr), tb.F32))
        ms = timed(core, 5)
        ms_layer = timed(lambda: mlayer.decode(hb, cb, lens, B, ctx * (CL + RP), ctx, comm=comm, out=lo), 5)
        byt = B * ctx * (CL + RP) * 2                       # the cache is replicated: every rank streams all of it
        mla.append({"ctx": ctx, "batch": B, "heads_per_gpu": H, "us": ms * 1e3, "layer_us": ms_layer * 1e3, "cache_bytes": byt,
                    "gbs_per_gpu": byt / ms / 1e6, "tflops": B * ctx * H * world * 2176.0 / ms / 1e9,
                    "frac_of_hbm_peak": byt / ms / 1e6 / peak_gbs})
        del cache
        torch.cuda.empty_cache()
    out["mla_dsv3_decode"] = mla
    mlayer.destroy()
    return out


# ----------------------------------------------------------------------------------------------
# --tofazen: the Tofazen family (bf16, dense) beside the Llama-shaped model (int4) at equal width, head and ffn sizes,
# random weights: decode and prefill throughput of both, and their like kernels one by one against their rooflines.
# ----------------------------------------------------------------------------------------------
TOFAZEN_SIZES = {
    # heads x 2 maps x dim = the Llama model's q width; vdim = its head size, so caches and products are equal
    "8b": {"layers": 32, "width": 4096, "heads": 32, "kv": 8, "dim": 64, "vdim": 128, "ff": 14336, "vocab": 128256},
    "1b": {"layers": 16, "width": 2048, "heads": 16, "kv": 4, "dim": 64, "vdim": 128, "ff": 8192, "vocab": 32000},
}


def build_tofazen(dev, tb, torch, stream, s, ctx, max_batch, window, keep_first):
    from tang_b200.tofazen import TofazenLayer, tensor_names

    gen = torch.Generator(device="cuda").manual_seed(5)
    layers = [TofazenLayer(s["heads"], s["kv"], s["dim"], s["vdim"], s["dim"] ** -0.5, 0.3, window, keep_first, None, s["ff"], 7.0)
              for _ in range(s["layers"])]
    cfg = tb.TofazenConfig(s["vocab"], s["width"], ctx + 1, 1e-6, 1.0, layers)
    model = tb.TofazenModel(dev, cfg, [0.5] * s["layers"], tb.BF16, max_batch, ctx + 1)
    d, qr, kr, vr = s["width"], s["heads"] * 2 * s["dim"], s["kv"] * 2 * s["dim"], s["kv"] * s["vdim"]
    shapes = {"embed": (s["vocab"], d), "pos": (ctx + 1, d), "final.norm": (1, d), "head": (s["vocab"], d), "norm1": (1, d), "q": (qr, d), "k": (kr, d),
              "v": (vr, d), "o": (d, s["heads"] * s["vdim"]), "gate": (s["ff"], d), "up": (s["ff"], d), "down": (d, s["ff"])}
    for name, tensor, layer in tensor_names(cfg):
        r, c = shapes[name if name in shapes else name.split(".")[-1]]
        with torch.cuda.stream(stream):
            t = (torch.randn((r, c), device="cuda", generator=gen) * (0.05 if r == 1 else c ** -0.5) + (1.0 if r == 1 else 0.0)).bfloat16()
        stream.synchronize()
        model.put_pointer(tensor, layer, t.data_ptr(), tb.BF16, r, c)
        del t
    return model


def run_tofazen(args) -> None:
    import ctypes as C

    import torch

    import tang_b200 as tb

    torch.cuda.set_device(0)
    dev = tb.QuantComputeDevice(0)
    L_ = dev._L
    stream = torch.cuda.ExternalStream(dev.stream, device=torch.device("cuda", 0))
    peaks = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json"))) if os.path.exists(os.path.join(ROOT, "MEASURED_PEAKS.json")) else {}
    hbm, tf = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    ctx = 2048
    sampler = ClockSampler(0)
    sampler.start()
    t_start = time.perf_counter()

    def graph_ms(fn, reps=10):
        fn()
        dev.sync()
        dev.begin_capture()
        fn()
        g = dev.end_capture()
        ms = _time_ms(torch, stream, dev, g.launch, reps, warm=3)
        g.free()
        return ms

    def rand_bf16(*shape, std=1.0):
        with torch.cuda.stream(stream):
            t = (torch.randn(shape, device="cuda") * std).bfloat16()
        stream.synchronize()
        return t

    def buf(t, dt):
        return tb.Buffer(dev, t.data_ptr(), t.numel(), dt, owns=False)

    out = {"metric": "tofazen_throughput", "unit": "tokens/s", "data": "synthetic", "dtype": "bf16", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf},
           "models": [], "kernels": []}
    batches = [1, 2, 4, 8, 16, 64]
    for size in [x for x in args.tofazen.split(",") if x in TOFAZEN_SIZES]:
        s = TOFAZEN_SIZES[size]
        c = {"d": s["width"], "n_heads": s["heads"], "n_kv": s["kv"], "hd": s["vdim"], "ffn": s["ff"], "vocab": s["vocab"], "ctx": ctx}
        w_layer = s["width"] * (s["heads"] * 2 * s["dim"] + s["kv"] * (2 * s["dim"] + s["vdim"]) + s["heads"] * s["vdim"] + 3 * s["ff"])
        params = s["layers"] * w_layer + s["vocab"] * s["width"]
        kv_row = s["layers"] * s["kv"] * (2 * s["dim"] + s["vdim"]) * 2
        for label, window, keep in (("full", ctx + 1, 0), ("window512", 512, 4)):
            model = build_tofazen(dev, tb, torch, stream, s, ctx, max(batches), window, keep)
            row = {"size": size, "model": "tofazen", "mask": label, "decode": {}, "prefill": {}}
            for B in batches:
                tok = dev.upload(np.random.randint(0, s["vocab"], B).astype(np.int32), tb.I32)
                pos = dev.upload(np.full(B, ctx, np.int32), tb.I32)
                lg = dev.alloc(B * s["vocab"], tb.F32)
                ms = graph_ms(lambda: model.decode(tok, pos, B, ctx + 1, lg))
                byt = params * 2 + B * kv_row * min(ctx + 1, window + keep)
                row["decode"][B] = {"ms": ms, "tokens_per_s": B / ms * 1e3, "frac_of_hbm": byt / ms / 1e6 / hbm}
            tok = dev.upload(np.random.randint(0, s["vocab"], ctx).astype(np.int32), tb.I32)
            cu, st = dev.upload(np.array([0, ctx], np.int32), tb.I32), dev.upload(np.zeros(1, np.int32), tb.I32)
            last, lg = dev.upload(np.array([ctx - 1], np.int32), tb.I32), dev.alloc(s["vocab"], tb.F32)
            ms = graph_ms(lambda: model.step(tok, ctx, cu, st, None, 1, ctx, ctx, last, 1, lg), 3)
            row["prefill"] = {"tokens": ctx, "ms": ms, "tokens_per_s": ctx / ms * 1e3, "frac_of_bf16": 2.0 * ctx * s["layers"] * w_layer / ms / 1e9 / tf}
            out["models"].append(row)
            model.destroy()
        if s["layers"] and not args.tofazen_only:
            torch.cuda.empty_cache()
            model = build_llama(dev, tb, torch, stream, None, 0, 1, s["layers"], max(batches), c)
            row = {"size": size, "model": "llama int4", "mask": "full", "decode": {}, "prefill": {}}
            q4 = params // 2 + params // 16
            for B in batches:
                tok = dev.upload(np.random.randint(0, s["vocab"], B).astype(np.int32), tb.I32)
                pos = dev.upload(np.full(B, ctx, np.int32), tb.I32)
                lg = dev.alloc(B * s["vocab"], tb.F32)
                ms = graph_ms(lambda: model.decode(tok, pos, B, ctx + 1, lg))
                row["decode"][B] = {"ms": ms, "tokens_per_s": B / ms * 1e3, "frac_of_hbm": (q4 + B * kv_row * (ctx + 1)) / ms / 1e6 / hbm}
            tok, st = dev.upload(np.random.randint(0, s["vocab"], ctx).astype(np.int32), tb.I32), dev.upload(np.zeros(1, np.int32), tb.I32)
            lg = dev.alloc(s["vocab"], tb.F32)
            model.prefill(tok, st, 1, ctx, lg)
            ms = _time_ms(torch, stream, dev, lambda: model.prefill(tok, st, 1, ctx, lg), 3)
            row["prefill"] = {"tokens": ctx, "ms": ms, "tokens_per_s": ctx / ms * 1e3, "frac_of_bf16": 2.0 * ctx * s["layers"] * w_layer / ms / 1e9 / tf}
            out["models"].append(row)
            model.destroy()
            torch.cuda.empty_cache()

    # ---- like kernels: a pass over several distinct weights (> L2), one launch each, from a graph
    def dense_handle(rows, cols):
        t = rand_bf16(rows, cols, std=cols ** -0.5)
        h = C.c_void_p()
        dev._check(L_.tq_dweight_create(dev._ctx, rows, cols, tb.BF16, C.byref(h)))
        dev._check(L_.tq_dweight_put(dev._ctx, h, C.c_void_p(t.data_ptr()), tb.BF16, rows, cols, 0, 0, 0))
        return h

    def q4_handle(rows, cols):
        with torch.cuda.stream(stream):
            pay = torch.randint(0, 256, (rows, cols // 2), dtype=torch.uint8, device="cuda")
            sc = (torch.rand((rows, cols // 32), device="cuda") * 0.018 + 0.002).half()
        stream.synchronize()
        h = C.c_void_p()
        dev._check(L_.tq_qweight_from_device_arrays(dev._ctx, tb.Q4_F16, C.c_void_p(pay.data_ptr()), C.c_void_p(sc.data_ptr()), rows, cols, C.byref(h)))
        dev.sync()
        return h

    for name, rows, cols in (("in", 34816, 4096), ("out", 4096, 18432)):
        n = 8
        dense, quant = [dense_handle(rows, cols) for _ in range(n)], [q4_handle(rows, cols) for _ in range(n)]
        for m in (1, 2, 4, 8, 16, 64, 256, 2048):
            x, y = rand_bf16(m, cols), torch.empty((m, rows), dtype=torch.bfloat16, device="cuda")
            stream.synchronize()
            xp, yp = C.c_void_p(x.data_ptr()), C.c_void_p(y.data_ptr())
            flops, io = 2.0 * m * rows * cols, m * (rows + cols) * 2
            for kind, hs, wb in (("dense bf16", dense, rows * cols * 2), ("int4", quant, rows * cols // 2 + rows * cols // 16)):
                if kind == "int4" and args.tofazen_only:
                    continue
                call = (lambda h: L_.tq_dlinear(dev._ctx, h, xp, cols, m, yp, tb.BF16, rows)) if hs is dense else \
                       (lambda h: L_.tq_qlinear(dev._ctx, h, xp, tb.BF16, 0, m, yp, tb.BF16, 0, None))
                us = graph_ms(lambda: [dev._check(call(h)) for h in hs]) / n * 1e3
                roof = max((wb + io) / hbm / 1e3, flops / tf / 1e6)
                out["kernels"].append({"kernel": f"linear {name} {rows}x{cols}", "kind": kind, "m": m, "us": us, "roofline_us": roof, "frac": roof / us})
        for h in dense:
            L_.tq_dweight_free(dev._ctx, h)
        for h in quant:
            L_.tq_qweight_free(dev._ctx, h)

    class Attn(C.Structure):
        _fields_ = [(k, C.c_uint32) for k in ("heads", "kv_heads", "dim", "vdim", "window", "keep_first")] + [
            (k, C.c_float) for k in ("scale", "lam", "out_scale", "eps")]

    H, G, D, V = 32, 8, 64, 128
    for B in (1, 16, 64):
        n = max(1, min(16, 64 // B * 2))               # distinct caches per pass
        k, v, q = rand_bf16(n, B, ctx, G * 2 * D), rand_bf16(n, B, ctx, G * V), rand_bf16(B, H * 2 * D)
        o = torch.empty((B, H * V), dtype=torch.bfloat16, device="cuda")
        lens = dev.upload(np.full(B, ctx, np.int32), tb.I32)
        rp = dev.upload(np.full(B, ctx - 1, np.int32), tb.I32)
        cr = dev.upload((np.arange(B) * ctx + ctx - 1).astype(np.int32), tb.I32)
        for kind, window in (("differential", ctx), ("differential window 512", 512), ("gqa", ctx)):
            a = Attn(H, G, D, V, window, 4, D ** -0.5, 0.5, 0.7, 1e-6)

            def one():
                for i in range(n):
                    if kind == "gqa":
                        dev._check(L_.tq_gqa_decode(dev._ctx, C.c_void_p(q.data_ptr()), C.c_void_p(k[i].data_ptr()), C.c_void_p(v[i].data_ptr()),
                                                    C.c_void_p(lens.ptr), B, H, G, 128, ctx * G * 128, ctx, C.c_void_p(o.data_ptr()), tb.BF16))
                    else:
                        dev._check(L_.tq_diff_attention(dev._ctx, C.byref(a), tb.BF16, C.c_void_p(q.data_ptr()), H * 2 * D, C.c_void_p(k[i].data_ptr()),
                                                        C.c_void_p(v[i].data_ptr()), B * ctx, None, C.c_void_p(rp.ptr), C.c_void_p(cr.ptr), B, B, 1, ctx,
                                                        C.c_void_p(o.data_ptr()), H * V))
            us = graph_ms(one) / n * 1e3
            roof = B * min(ctx, window + (4 if window < ctx else 0)) * G * (2 * D + V) * 2 / hbm / 1e3
            out["kernels"].append({"kernel": "decode attention", "kind": kind, "m": B, "us": us, "roofline_us": roof, "frac": roof / us})
        del k, v
        torch.cuda.empty_cache()
    for T in (512, 2048):
        k, v, q = rand_bf16(T, G * 2 * D), rand_bf16(T, G * V), rand_bf16(T, H * 2 * D)
        o = torch.empty((T, H * V), dtype=torch.bfloat16, device="cuda")
        cu, st = dev.upload(np.array([0, T], np.int32), tb.I32), dev.upload(np.zeros(1, np.int32), tb.I32)
        rp = dev.upload(np.arange(T, dtype=np.int32), tb.I32)
        for kind, window in (("differential", T), ("differential window 256", 256), ("gqa", T)):
            a = Attn(H, G, D, V, window, 4, D ** -0.5, 0.5, 0.7, 1e-6)
            if kind == "gqa":
                fn = lambda: dev._check(L_.tq_gqa_prefill(dev._ctx, C.c_void_p(q.data_ptr()), C.c_void_p(k.data_ptr()), C.c_void_p(v.data_ptr()),
                                                          C.c_void_p(st.ptr), 1, T, H, G, 128, T * G * 128, C.c_void_p(o.data_ptr()), tb.BF16))
                flops = 4.0 * H * 128 * T * (T + 1) / 2
            else:
                fn = lambda: dev._check(L_.tq_diff_attention(dev._ctx, C.byref(a), tb.BF16, C.c_void_p(q.data_ptr()), H * 2 * D, C.c_void_p(k.data_ptr()),
                                                             C.c_void_p(v.data_ptr()), T, C.c_void_p(cu.ptr), C.c_void_p(rp.ptr), C.c_void_p(rp.ptr), 1, T, T, T,
                                                             C.c_void_p(o.data_ptr()), H * V))
                pairs = sum(min(i + 1, window + 4) for i in range(T))
                flops = 2.0 * H * 2 * (D + V) * pairs
            us = graph_ms(fn) * 1e3
            out["kernels"].append({"kernel": "prefill attention", "kind": kind, "m": T, "us": us, "tflops": flops / us / 1e6, "roofline_us": flops / tf / 1e6,
                                   "frac": flops / tf / 1e6 / us})
    out["clocks"] = sampler.stop(t_start, time.perf_counter())
    print(json.dumps(out))

# ----------------------------------------------------------------------------------------------
# --numuzen: the Numuzen family (bf16) beside the Tofazen family at equal width, head sizes, window and active feed-forward,
# random weights: decode and prefill throughput of both, and the kernels one by one against their rooflines.
# ----------------------------------------------------------------------------------------------
NUMUZEN_SIZES = {
    # alternating mixers; top experts of ff values together are as wide as the dense model's feed-forward
    "8b": {"layers": 32, "width": 4096, "heads": 32, "kv": 8, "dim": 128, "gla": (16, 128, 256), "experts": 8, "top": 2, "ff": 7168, "vocab": 128256},
    "1b": {"layers": 16, "width": 2048, "heads": 16, "kv": 4, "dim": 128, "gla": (8, 128, 256), "experts": 32, "top": 4, "ff": 2048, "vocab": 32000},
}


def build_numuzen(dev, tb, torch, stream, s, max_seq, max_batch, window):
    from tang_b200 import numuzen as nz

    gen = torch.Generator(device="cuda").manual_seed(7)
    experts = nz.Experts(s["experts"], s["top"], s["ff"], 7.0)
    rot = nz.Rotation(64, 500000.0, 4.0, 4096, 32.0, 1.0)
    gh, gd, gv = s["gla"]
    layers = [nz.NumuzenLayer(nz.ATTENTION, s["heads"], s["dim"], s["dim"], s["dim"] ** -0.5, s["kv"], window, 50.0, rot, experts=experts) if i % 2 == 0 else
              nz.NumuzenLayer(nz.GLA, gh, gd, gv, gd ** -0.5, tau=16.0, rank=16, experts=experts) for i in range(s["layers"])]
    cfg = tb.NumuzenConfig(s["vocab"], s["width"], 1e-6, layers)
    model = tb.NumuzenModel(dev, cfg, tb.BF16, max_batch, max_seq)
    pool = {}
    for name, tensor, i, e in nz.tensor_names(cfg):
        l, d = cfg.layers[i], s["width"]
        qr, vr, kr = l.heads * l.dim, l.heads * l.vdim, (l.kv_heads or l.heads) * l.dim
        r, c = {nz.EMBED: (s["vocab"], d), nz.Q: (qr, d), nz.K: (kr, d), nz.V: (vr, d), nz.G: (vr, d), nz.O: (d, vr), nz.Q_NORM: (1, qr), nz.K_NORM: (1, kr),
                nz.O_NORM: (1, l.vdim), nz.A1: (l.rank, d), nz.A2: (qr, l.rank), nz.A2_BIAS: (1, qr), nz.ROUTER: (s["experts"], d), nz.GATE: (s["ff"], d),
                nz.UP: (s["ff"], d), nz.DOWN: (d, s["ff"])}.get(tensor, (1, d))
        plain = tensor in (nz.Q_NORM, nz.K_NORM, nz.O_NORM)
        key = (r, c, plain, tensor in (nz.ROUTER,) and i)
        if key not in pool:
            with torch.cuda.stream(stream):
                pool[key] = (torch.randn((r, c), device="cuda", generator=gen) * (0.05 if r == 1 else c ** -0.5) + (1.0 if plain else 0.0)).bfloat16()
            stream.synchronize()
        model.put_pointer(tensor, i, pool[key].data_ptr(), tb.BF16, r, c, e)
    return model


def run_numuzen(args) -> None:
    import ctypes as C

    import torch

    import tang_b200 as tb

    torch.cuda.set_device(0)
    dev = tb.QuantComputeDevice(0)
    L_ = dev._L
    stream = torch.cuda.ExternalStream(dev.stream, device=torch.device("cuda", 0))
    peaks = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json"))) if os.path.exists(os.path.join(ROOT, "MEASURED_PEAKS.json")) else {}
    hbm, tf = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    ctx, window = 2048, 512
    sampler = ClockSampler(0)
    sampler.start()
    t_start = time.perf_counter()

    def graph_ms(fn, reps=10):
        fn()
        dev.sync()
        dev.begin_capture()
        fn()
        g = dev.end_capture()
        ms = _time_ms(torch, stream, dev, g.launch, reps, warm=3)
        g.free()
        return ms

    def rand(*shape, std=1.0, dt=None):
        with torch.cuda.stream(stream):
            t = torch.randn(shape, device="cuda") * std
            t = t if dt == tb.F32 else t.bfloat16()
        stream.synchronize()
        return t

    P = lambda t: C.c_void_p(t.data_ptr() if hasattr(t, "data_ptr") else t.ptr)
    ints = lambda a: dev.upload(np.asarray(a, np.int32).reshape(-1), tb.I32)

    def touched(experts, top, rows):
        """Expected number of experts that `rows` rows choose."""
        return experts * (1 - (1 - top / experts) ** rows)

    out = {"metric": "numuzen_throughput", "unit": "tokens/s", "data": "synthetic", "dtype": "bf16", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf},
           "window": window, "models": [], "kernels": []}
    batches = [1, 2, 4, 8, 16, 64]

    def time_model(size, name, model, s, decode_bytes, prefill_params):
        row = {"size": size, "model": name, "decode": {}, "prefill": {}}
        for B in batches:
            tok = ints(np.random.randint(0, s["vocab"], B))
            pos, lg = ints(np.full(B, ctx)), dev.alloc(B * s["vocab"], tb.F32)
            ms = graph_ms(lambda: model.decode(tok, pos, B, ctx + 1, lg))
            row["decode"][B] = {"ms": ms, "tokens_per_s": B / ms * 1e3, "frac_of_hbm": decode_bytes(B) / ms / 1e6 / hbm}
        tok = ints(np.random.randint(0, s["vocab"], ctx))
        cu, st, last, lg = ints([0, ctx]), ints([0]), ints([ctx - 1]), dev.alloc(s["vocab"], tb.F32)
        ms = graph_ms(lambda: model.step(tok, ctx, cu, st, None, 1, ctx, ctx, last, 1, lg), 3)
        row["prefill"] = {"tokens": ctx, "ms": ms, "tokens_per_s": ctx / ms * 1e3, "frac_of_bf16": 2.0 * ctx * prefill_params / ms / 1e9 / tf}
        out["models"].append(row)
        model.destroy()
        torch.cuda.empty_cache()

    for size in [x for x in args.numuzen.split(",") if x in NUMUZEN_SIZES]:
        s = NUMUZEN_SIZES[size]
        d, (gh, gd, gv) = s["width"], s["gla"]
        att = d * (3 * s["heads"] + s["kv"]) * s["dim"]
        rec = d * (2 * gh * gd + 3 * gh * gv + 16)
        mixers = s["layers"] // 2 * (att + rec)
        one = 3 * d * s["ff"]
        kv = s["layers"] // 2 * s["kv"] * 2 * s["dim"] * 2 * window
        state = s["layers"] // 2 * gh * gd * gv * 4 * 2
        fixed = 2 * (mixers + s["layers"] * s["experts"] * d + s["vocab"] * d)
        time_model(size, "numuzen", build_numuzen(dev, tb, torch, stream, s, ctx + 1, max(batches), window), s,
                   lambda B: fixed + 2 * s["layers"] * one * touched(s["experts"], s["top"], B) + B * (kv + state), mixers + s["layers"] * s["top"] * one)
        if not args.numuzen_only:
            z = dict(TOFAZEN_SIZES[size])
            w = z["width"] * (z["heads"] * 2 * z["dim"] + z["kv"] * (2 * z["dim"] + z["vdim"]) + z["heads"] * z["vdim"] + 3 * z["ff"])
            row_b = z["layers"] * z["kv"] * (2 * z["dim"] + z["vdim"]) * 2
            time_model(size, "tofazen", build_tofazen(dev, tb, torch, stream, z, ctx, max(batches), window, 4), z,
                       lambda B: 2 * (z["layers"] * w + z["vocab"] * z["width"]) + B * row_b * (window + 4), z["layers"] * w)

    def kernel(name, m, us, byt=0.0, flops=0.0):
        roof = max(byt / hbm / 1e3, flops / tf / 1e6)
        out["kernels"].append({"kernel": name, "m": m, "us": round(us, 2), "roofline_us": round(roof, 2), "frac": round(roof / us, 3)})

    # ---- linear layers: the mixers' projections, and the experts beside a dense layer of the same products
    def handle(rows, cols):
        t = rand(min(rows, 65536), cols, std=cols ** -0.5)
        h = C.c_void_p()
        dev._check(L_.tq_dweight_create(dev._ctx, rows, cols, tb.BF16, C.byref(h)))
        for r in range(0, rows, 65536):
            n = min(65536, rows - r)
            dev._check(L_.tq_dweight_put(dev._ctx, h, P(t), tb.BF16, n, cols, r, 0, 0))
        return h

    d = 4096
    for name, rows, cols in (("attention in", 9216, d), ("recurrent in", 12304, d), ("mixer out", d, 4096)):
        hs = [handle(rows, cols) for _ in range(8)]
        for m in (1, 8, 64, 2048):
            x, y = rand(m, cols), torch.empty((m, rows), dtype=torch.bfloat16, device="cuda")
            us = graph_ms(lambda: [dev._check(L_.tq_dlinear(dev._ctx, h, P(x), cols, m, P(y), tb.BF16, rows)) for h in hs]) / len(hs) * 1e3
            kernel(f"linear {name} {rows}x{cols}", m, us, rows * cols * 2 + m * (rows + cols) * 2, 2.0 * m * rows * cols)
        for h in hs:
            L_.tq_dweight_free(dev._ctx, h)
    for E, top, ff, d in ((8, 2, 7168, 4096), (32, 4, 2048, 2048)):
        n = 2
        gu, dn = [handle(E * 2 * ff, d) for _ in range(n)], [handle(E * d, ff) for _ in range(n)]
        dense_gu, dense_dn = [handle(top * 2 * ff, d) for _ in range(3 * n)], [handle(d, top * ff) for _ in range(3 * n)]
        rng = np.random.default_rng(0)
        for m in (1, 2, 4, 8, 16, 64, 256, 2048):
            pairs = m * top
            chosen = np.stack([rng.permutation(E)[:top] for _ in range(m)])
            counts = np.bincount(chosen.reshape(-1), minlength=E)
            chunk = L_.tq_dense_group_chunk(tb.BF16, max(d, ff), pairs, E)
            jobs, first = [], 0
            for e in range(E):
                jobs += [(e, first + i, min(chunk, counts[e] - i), 0) for i in range(0, counts[e], chunk)]
                first += counts[e]
            jd, nd = ints(jobs), ints([len(jobs)])
            sr = ints(np.argsort(chosen.reshape(-1), kind="stable") // top) if chunk <= 8 else None
            w = dev.upload(np.ones(pairs, np.float32), tb.F32)
            mj = min(pairs, E + pairs // chunk)
            x, act, y = rand(max(pairs, m), d), torch.empty((pairs, ff), dtype=torch.bfloat16, device="cuda"), torch.empty((pairs, d), device="cuda")
            null = C.c_void_p(0)
            live = int((counts > 0).sum())
            for what, hs, call, wb, io in (
                    ("gate/up", gu, lambda h: L_.tq_dlinear_grouped(dev._ctx, h, P(x), d, pairs, P(jd), P(nd), mj, chunk, 2 * ff, P(sr) if sr else null, P(w), 7.0, 1.702,
                                                                    P(act), tb.BF16, ff), live * 2 * ff * d * 2, pairs * (d + ff) * 2),
                    ("down", dn, lambda h: L_.tq_dlinear_grouped(dev._ctx, h, P(act), ff, pairs, P(jd), P(nd), mj, chunk, d, null, null, 0.0, 0.0, P(y), tb.F32, d),
                     live * ff * d * 2, pairs * (ff * 2 + d * 4))):
                us = graph_ms(lambda: [dev._check(call(h)) for h in hs]) / len(hs) * 1e3
                kernel(f"experts {what} {E}x{ff}x{d} top {top}", m, us, wb + io, 2.0 * pairs * ff * d * (2 if what == "gate/up" else 1))
            dx, dy = rand(m, max(d, top * ff)), torch.empty((m, max(d, top * 2 * ff)), device="cuda")
            for what, hs, rows, cols in (("gate/up", dense_gu, top * 2 * ff, d), ("down", dense_dn, d, top * ff)):
                us = graph_ms(lambda: [dev._check(L_.tq_dlinear(dev._ctx, h, P(dx), cols, m, P(dy), tb.BF16 if what == "gate/up" else tb.F32, rows)) for h in hs]) / len(hs) * 1e3
                kernel(f"dense {what} {rows}x{cols}", m, us, rows * cols * 2 + m * (cols * 2 + rows * (2 if what == "gate/up" else 4)), 2.0 * m * rows * cols)
        for h in gu + dn + dense_gu + dense_dn:
            L_.tq_dweight_free(dev._ctx, h)
        del x, act, y, dx, dy
        torch.cuda.empty_cache()

    # ---- attention and recurrence, one row per sequence at position ctx - 1, then one prompt
    class Win(C.Structure):
        _fields_ = [(k, C.c_uint32) for k in ("heads", "kv_heads", "dim", "vdim", "window")] + [(k, C.c_float) for k in ("scale", "softcap", "sink")]

    class Diff(C.Structure):
        _fields_ = [(k, C.c_uint32) for k in ("heads", "kv_heads", "dim", "vdim", "window", "keep_first")] + [
            (k, C.c_float) for k in ("scale", "lam", "out_scale", "eps")]

    class Gla(C.Structure):
        _fields_ = [(k, C.c_uint32) for k in ("heads", "dim", "vdim", "rank")] + [(k, C.c_float) for k in ("tau", "q_scale", "eps")]

    H, G, D = 32, 8, 128
    gh, gd, gv = 16, 128, 256
    gw = 2 * gh * gd + 2 * gh * gv
    a2, bias, gnorm = rand(gh * gd, 16, dt=tb.F32), rand(gh * gd, dt=tb.F32), rand(gv, dt=tb.F32)

    def attention(kind, w, q, k, v, gate, o, B, rows, n_seqs, cu, rp, cr, max_q):
        if kind == "window":
            a = Win(H, G, D, D, w, D ** -0.5, 50.0, 0.0)
            return L_.tq_window_attention(dev._ctx, C.byref(a), tb.BF16, P(q), H * D, P(gate), H * D, P(k), P(v), B * ctx, cu, P(rp), P(cr), n_seqs, rows, max_q, ctx,
                                          P(o), H * D)
        a = Diff(H, G, D // 2, D, w, 4, D ** -0.5, 0.5, 0.7, 1e-6)
        return L_.tq_diff_attention(dev._ctx, C.byref(a), tb.BF16, P(q), H * D, P(k), P(v), B * ctx, cu, P(rp), P(cr), n_seqs, rows, max_q, ctx, P(o), H * D)

    def recurrence(x, a1, state, o, rows, n_seqs, cu, rp, cr, max_q):
        g, off = Gla(gh, gd, gv, 16, 16.0, gd ** -0.5, 1e-6), lambda n: C.c_void_p(x.data_ptr() + 2 * n)
        return L_.tq_gla(dev._ctx, C.byref(g), tb.BF16, off(0), off(gh * gd), off(2 * gh * gd), off(2 * gh * gd + gh * gv), gw, P(a1), 16, P(a2), P(bias), P(gnorm),
                         P(state), ctx, n_seqs * ctx, cu, P(rp), P(cr), n_seqs, rows, max_q, P(o), gh * gv)

    null = C.c_void_p(0)
    for B in (1, 16, 64):
        n = max(1, min(16, 64 // B * 2))               # distinct caches per pass
        k, v, q, gate = rand(n, B, ctx, G * D), rand(n, B, ctx, G * D), rand(B, H * D), rand(B, H * D)
        o = torch.empty((B, H * D), dtype=torch.bfloat16, device="cuda")
        rp, cr = ints(np.full(B, ctx - 1)), ints(np.arange(B) * ctx + ctx - 1)
        for kind in ("window", "differential"):
            for w in (window, ctx):
                us = graph_ms(lambda: [dev._check(attention(kind, w, q, k[i], v[i], gate, o, B, B, B, null, rp, cr, 1)) for i in range(n)]) / n * 1e3
                kernel(f"decode attention {kind} {w}", B, us, B * w * G * D * 2 * 2)
        del k, v
        st = [rand(B, gh, gd, gv, dt=tb.F32) for _ in range(max(4, min(64, 128 // B)))]
        x, a1, o = rand(B, gw), rand(B, 16, dt=tb.F32), torch.empty((B, gh * gv), dtype=torch.bfloat16, device="cuda")
        us = graph_ms(lambda: [dev._check(recurrence(x, a1, t, o, B, B, null, rp, cr, 1)) for t in st]) / len(st) * 1e3
        kernel("decode recurrence", B, us, B * gh * gd * gv * 4 * 2)
        del st
        torch.cuda.empty_cache()
    for T in (512, 2048):
        k, v, q, gate = rand(T, G * D), rand(T, G * D), rand(T, H * D), rand(T, H * D)
        o = torch.empty((T, H * D), dtype=torch.bfloat16, device="cuda")
        cu, rp = ints([0, T]), ints(np.arange(T))
        for kind in ("window", "differential"):
            for w in (256, ctx):
                us = graph_ms(lambda: dev._check(attention(kind, w, q, k, v, gate, o, 1, T, 1, P(cu), rp, rp, T))) * 1e3
                kernel(f"prefill attention {kind} {w}", T, us, 0, 2.0 * H * (2 * D if kind == "window" else 3 * D) * sum(min(i + 1, w) for i in range(T)))
        x, a1, st = rand(T, gw), rand(T, 16, dt=tb.F32), rand(1, gh, gd, gv, dt=tb.F32)
        o = torch.empty((T, gh * gv), dtype=torch.bfloat16, device="cuda")
        us = graph_ms(lambda: dev._check(recurrence(x, a1, st, o, T, 1, P(cu), rp, rp, T))) * 1e3
        # (chunked form with single products: 64-token pair weights and their values, contributions to and readings of the state)
        kernel("prefill recurrence", T, us, T * (gw + gh * gv) * 2, 2.0 * T * gh * (32 * (gd + gv) + 2 * gd * gv))

    # ---- row operators beside the plain norm
    for m in (1, 64, 2048):
        x, y, gain, h = rand(m, 4096, dt=tb.F32), rand(m * 2, 4096, dt=tb.F32), rand(4096, dt=tb.F32), torch.empty((m, 4096), dtype=torch.bfloat16, device="cuda")
        slots = ints(np.random.permutation(2 * m))
        n = 20
        for name, call, byt in (
                ("post-norm, stream, next norm", lambda: L_.tq_add_norm(dev._ctx, P(x), P(y), null, 1, P(gain), P(gain), m, 4096, 1e-6, P(h), tb.BF16, 4096), m * 4096 * 14),
                ("the same over two experts", lambda: L_.tq_add_norm(dev._ctx, P(x), P(y), P(slots), 2, P(gain), P(gain), m, 4096, 1e-6, P(h), tb.BF16, 4096), m * 4096 * 18),
                ("plain norm", lambda: L_.tq_rms_norm(dev._ctx, P(x), tb.F32, null, P(gain), tb.F32, m, 4096, 1e-6, P(h), tb.BF16, null), m * 4096 * 6)):
            kernel(name, m, graph_ms(lambda: [dev._check(call()) for _ in range(n)]) / n * 1e3, byt)
        q, raw, keys, qg, kg, fr = rand(m, H * D), rand(m, G * D), rand(m, G * D), rand(H * D), rand(G * D), rand(32, dt=tb.F32)
        rp = ints(np.arange(m))
        us = graph_ms(lambda: [dev._check(L_.tq_qk_norm_rope(dev._ctx, tb.BF16, H, G, D, P(q), H * D, P(raw), P(keys), m, P(qg), P(kg), 64, P(fr), 1.0, 1e-6, P(rp), P(rp), m))
                               for _ in range(n)]) / n * 1e3
        kernel("query/key norm and rotation", m, us, m * (H + G) * D * 4)
        z = rand(m, 32, dt=tb.F32)
        bufs = [ints(np.zeros(m * 4)) for _ in range(4)] + [ints(np.zeros(4 * (m * 4 + 32))), ints([0])]
        us = graph_ms(lambda: [dev._check(L_.tq_route(dev._ctx, P(z), m, 32, 4, 0, 0, 8, *map(P, bufs))) for _ in range(n)]) / n * 1e3
        kernel("routing, 4 of 32", m, us, m * 32 * 4)
    out["clocks"] = sampler.stop(t_start, time.perf_counter())
    print(json.dumps(out))


# ----------------------------------------------------------------------------------------------
# --dotanex: the Dotanex family (bf16) beside the Numuzen family at equal width, head sizes, window and active feed-forward,
# random weights: decode and prefill throughput of both, and the new kernels beside the like ones, against their rooflines.
# ----------------------------------------------------------------------------------------------
DOTANEX_SIZES = {
    # of four layers: attention, lightning, latent attention, lightning; of `top` choices two thirds (8b) or four fifths (1b) fall on
    # experts with weights, which together with the shared one are as wide as the other models' feed-forward
    "8b": {**{k: NUMUZEN_SIZES["8b"][k] for k in ("layers", "width", "heads", "kv", "dim", "vocab")}, "lightning": (16, 128, 256), "latent": (1536, 512, 64),
           "experts": 8, "identity": 4, "top": 3, "ff": 4096, "shared": 6144, "streams": 4},
    "1b": {**{k: NUMUZEN_SIZES["1b"][k] for k in ("layers", "width", "heads", "kv", "dim", "vocab")}, "lightning": (8, 128, 256), "latent": (768, 512, 64),
           "experts": 32, "identity": 8, "top": 5, "ff": 1536, "shared": 2048, "streams": 4},
}


def build_dotanex(dev, tb, torch, stream, s, max_seq, max_batch, window):
    from tang_b200 import dotanex as dx

    gen = torch.Generator(device="cuda").manual_seed(7)
    mlp = dx.FeedForward(dx.MOE, s["ff"], s["experts"], s["identity"], s["top"], 7.0, s["shared"], 7.0)
    (lh, ld, lv), (q_rank, kv_rank, rot) = s["lightning"], s["latent"]
    banded = dx.Rotation(64, 500000.0, 4.0, 4096, low=1.0, high=4.0)
    yarn = dx.Rotation(rot, 500000.0, 4.0, 4096, fast=32.0, slow=1.0)
    kinds = [dx.DotanexLayer(dx.ATTENTION, s["heads"], s["dim"], s["dim"], s["dim"] ** -0.5, s["kv"], window, banded, mlp=mlp),
             dx.DotanexLayer(dx.LIGHTNING, lh, ld, lv, decay=tuple(1 - 2.0 ** (-2 - 0.3 * h) for h in range(lh)), mlp=mlp),
             dx.DotanexLayer(dx.LATENT, s["heads"], s["dim"], s["dim"], (s["dim"] + rot) ** -0.5, rot=yarn, q_rank=q_rank, kv_rank=kv_rank, rot_dim=rot, mlp=mlp)]
    cfg = tb.DotanexConfig(s["vocab"], s["width"], s["streams"], 1e-6, [kinds[(0, 1, 2, 1)[i % 4]] for i in range(s["layers"])])
    model = tb.DotanexModel(dev, cfg, tb.BF16, max_batch, max_seq)
    d, S, n = s["width"], s["streams"], s["experts"] + s["identity"]
    pool = {}
    for name, tensor, i, e in dx.tensor_names(cfg):
        l = cfg.layers[i]
        H, G, D, V = l.heads, l.kv_heads or l.heads, l.dim, l.vdim
        r, c = {dx.EMBED: (s["vocab"], d), dx.HEAD: (s["vocab"], d), dx.HC1_IN: (1, S), dx.HC2_IN: (1, S), dx.HC1_OUT: (1, S), dx.HC2_OUT: (1, S), dx.HC1_MIX: (S, S),
                dx.HC2_MIX: (S, S), dx.Q: (H * D, d), dx.K: (G * D, d), dx.V: (H * V, d), dx.G: (H * V, d), dx.O: (d, H * V), dx.Q_NORM: (1, D), dx.K_NORM: (1, D),
                dx.SINK: (1, H), dx.O_NORM: (1, H * V), dx.DQ: (q_rank, d), dx.DQ_NORM: (1, q_rank), dx.UQ: (H * (D + rot), q_rank), dx.DKV: (kv_rank + rot, d),
                dx.DKV_NORM: (1, kv_rank), dx.UK: (H * D, kv_rank), dx.UV: (H * V, kv_rank), dx.ROUTER: (n, d), dx.CORRECTION: (1, n), dx.GATE: (s["ff"], d),
                dx.UP: (s["ff"], d), dx.DOWN: (d, s["ff"]), dx.SHARED_GATE: (s["shared"], d), dx.SHARED_UP: (s["shared"], d),
                dx.SHARED_DOWN: (d, s["shared"])}.get(tensor, (1, d))
        level = {dx.HC1_IN: 1.0 / S, dx.HC2_IN: 1.0 / S, dx.HC1_OUT: 0.5, dx.HC2_OUT: 0.5, dx.HC1_MIX: 1.0 / S, dx.HC2_MIX: 1.0 / S, dx.SINK: 0.0, dx.CORRECTION: 0.0}.get(
            tensor, 1.0 if r == 1 else 0.0)
        key = (r, c, level, tensor == dx.ROUTER and i)
        if key not in pool:
            with torch.cuda.stream(stream):
                pool[key] = (torch.randn((r, c), device="cuda", generator=gen) * (0.02 if r == 1 or r == S else c ** -0.5) + level).bfloat16()
            stream.synchronize()
        model.put_pointer(tensor, i, pool[key].data_ptr(), tb.BF16, r, c, e)
    return model


def run_dotanex(args) -> None:
    import ctypes as C

    import torch

    import tang_b200 as tb

    torch.cuda.set_device(0)
    dev = tb.QuantComputeDevice(0)
    L_ = dev._L
    stream = torch.cuda.ExternalStream(dev.stream, device=torch.device("cuda", 0))
    peaks = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json"))) if os.path.exists(os.path.join(ROOT, "MEASURED_PEAKS.json")) else {}
    hbm, tf = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    ctx, window = 2048, 512
    sampler = ClockSampler(0)
    sampler.start()
    t_start = time.perf_counter()

    def graph_ms(fn, reps=10):
        fn()
        dev.sync()
        dev.begin_capture()
        fn()
        g = dev.end_capture()
        ms = _time_ms(torch, stream, dev, g.launch, reps, warm=3)
        g.free()
        return ms

    def rand(*shape, std=1.0, dt=None):
        with torch.cuda.stream(stream):
            t = torch.randn(shape, device="cuda") * std
            t = t if dt == tb.F32 else t.bfloat16()
        stream.synchronize()
        return t

    P = lambda t: C.c_void_p(t.data_ptr() if hasattr(t, "data_ptr") else t.ptr)
    ints = lambda a: dev.upload(np.asarray(a, np.int32).reshape(-1), tb.I32)
    null = C.c_void_p(0)
    touched = lambda experts, share, rows: experts * (1 - (1 - share) ** rows)      # expected number of experts that `rows` rows choose
    out = {"metric": "dotanex_throughput", "unit": "tokens/s", "data": "synthetic", "dtype": "bf16", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf},
           "window": window, "models": [], "kernels": []}
    batches = [1, 2, 4, 8, 16, 64]

    def time_model(size, name, model, s, decode_bytes, prefill_flops):
        row = {"size": size, "model": name, "decode": {}, "prefill": {}}
        for B in batches:
            tok = ints(np.random.randint(0, s["vocab"], B))
            pos, lg = ints(np.full(B, ctx)), dev.alloc(B * s["vocab"], tb.F32)
            ms = graph_ms(lambda: model.decode(tok, pos, B, ctx + 1, lg))
            row["decode"][B] = {"ms": ms, "tokens_per_s": B / ms * 1e3, "frac_of_hbm": decode_bytes(B) / ms / 1e6 / hbm}
        for T in (512, ctx):
            tok = ints(np.random.randint(0, s["vocab"], T))
            cu, st, last, lg = ints([0, T]), ints([0]), ints([T - 1]), dev.alloc(s["vocab"], tb.F32)
            ms = graph_ms(lambda: model.step(tok, T, cu, st, None, 1, T, T, last, 1, lg), 3)
            row["prefill"][T] = {"ms": ms, "tokens_per_s": T / ms * 1e3, "frac_of_bf16": T * prefill_flops(T) / ms / 1e9 / tf}
        out["models"].append(row)
        model.destroy()
        torch.cuda.empty_cache()

    for size in [x for x in args.dotanex.split(",") if x in DOTANEX_SIZES]:
        s = DOTANEX_SIZES[size]
        d, H, D, (lh, ld, lv), (qr, kr, rot) = s["width"], s["heads"], s["dim"], s["lightning"], s["latent"]
        n = s["experts"] + s["identity"]
        att = d * (2 * H + s["kv"]) * D
        rec = d * (2 * lh * ld + 3 * lh * lv)
        lat = d * (qr + kr + rot + 2 * H * D) + qr * H * (D + rot) + 2 * kr * H * D
        mixers = s["layers"] // 4 * (att + 2 * rec + lat)
        one, share = 3 * d * s["ff"], s["top"] / n
        fixed = 2 * (mixers + s["layers"] * (n * d + 3 * d * s["shared"]) + s["vocab"] * d)
        per_row = s["layers"] // 4 * (s["kv"] * 2 * D * 2 * window + 2 * lh * ld * lv * 4 * 2 + (kr + rot) * 2 * ctx)
        active = mixers + s["layers"] * (s["experts"] * share * one + 3 * d * s["shared"])
        time_model(size, "dotanex", build_dotanex(dev, tb, torch, stream, s, ctx + 1, max(batches), window), s,
                   lambda B: fixed + 2 * s["layers"] * one * touched(s["experts"], share, B) + B * per_row,
                   lambda T: 2.0 * active + s["layers"] // 4 * H * T * (2 * D + rot))
        if not args.dotanex_only:
            z = NUMUZEN_SIZES[size]
            gh, gd, gv = z["gla"]
            zm = z["layers"] // 2 * (d * (3 * H + z["kv"]) * D + d * (2 * gh * gd + 3 * gh * gv + 16))
            zone, zrow = 3 * d * z["ff"], z["layers"] // 2 * (z["kv"] * 2 * D * 2 * window + gh * gd * gv * 8)
            time_model(size, "numuzen", build_numuzen(dev, tb, torch, stream, z, ctx + 1, max(batches), window), z,
                       lambda B: 2 * (zm + z["layers"] * z["experts"] * d + z["vocab"] * d + z["layers"] * zone * touched(z["experts"], z["top"] / z["experts"], B)) + B * zrow,
                       lambda T: 2.0 * (zm + z["layers"] * z["top"] * zone))

    def kernel(name, m, us, byt=0.0, flops=0.0):
        roof = max(byt / hbm / 1e3, flops / tf / 1e6)
        out["kernels"].append({"kernel": name, "m": m, "us": round(us, 2), "roofline_us": round(roof, 2), "frac": round(roof / us, 3)})

    # ---- decode: absorbed latent attention beside the int8 family's, lightning beside the gated recurrence
    class Win(C.Structure):
        _fields_ = [(k, C.c_uint32) for k in ("heads", "kv_heads", "dim", "vdim", "window")] + [(k, C.c_float) for k in ("scale", "softcap", "sink")]

    class Gla(C.Structure):
        _fields_ = [(k, C.c_uint32) for k in ("heads", "dim", "vdim", "rank")] + [(k, C.c_float) for k in ("tau", "q_scale", "eps")]

    def handle(rows, cols):
        t, h = rand(min(rows, 65536), cols, std=cols ** -0.5), C.c_void_p()
        dev._check(L_.tq_dweight_create(dev._ctx, rows, cols, tb.BF16, C.byref(h)))
        for r in range(0, rows, 65536):
            dev._check(L_.tq_dweight_put(dev._ctx, h, P(t), tb.BF16, min(65536, rows - r), cols, r, 0, 0))
        return h

    H, D, R, K = 32, 128, 64, 512
    lh, ld, lv = 16, 128, 256
    width = 2 * lh * ld + 2 * lh * lv
    freq, decay = rand(R // 2, dt=tb.F32), torch.full((lh,), 0.97, device="cuda")
    norm, gnorm, a2, bias = rand(lh * lv, dt=tb.F32), rand(lv, dt=tb.F32), rand(lh * ld, 16, dt=tb.F32), rand(lh * ld, dt=tb.F32)
    torch.cuda.synchronize()

    def lightning(x, st, o, rows, n_seqs, cu, rp, cr, max_q):
        off = lambda c: C.c_void_p(x.data_ptr() + 2 * c)
        return L_.tq_lightning(dev._ctx, tb.BF16, lh, ld, lv, 1e-6, P(decay), off(0), off(lh * ld), off(2 * lh * ld), off(2 * lh * ld + lh * lv), width, P(norm), P(st), ctx,
                               n_seqs * ctx, cu, P(rp), P(cr), n_seqs, rows, max_q, P(o), lh * lv)

    def recurrence(x, a1, st, o, rows, n_seqs, cu, rp, cr, max_q):
        g, off = Gla(lh, ld, lv, 16, 16.0, ld ** -0.5, 1e-6), lambda c: C.c_void_p(x.data_ptr() + 2 * c)
        return L_.tq_gla(dev._ctx, C.byref(g), tb.BF16, off(0), off(lh * ld), off(2 * lh * ld), off(2 * lh * ld + lh * lv), width, P(a1), 16, P(a2), P(bias), P(gnorm),
                         P(st), ctx, n_seqs * ctx, cu, P(rp), P(cr), n_seqs, rows, max_q, P(o), lh * lv)

    uk, uv = [handle(H * K, D) for _ in range(16)], [handle(H * D, K) for _ in range(16)]
    q8 = []
    for _ in range(16):
        with torch.cuda.stream(stream):
            wk, wv = (torch.randint(-127, 128, (H * r, c), dtype=torch.int8, device="cuda") for r, c in ((K, D), (D, K)))
            sk, sv = (torch.full((H * r,), 0.002, device="cuda") for r in (K, D))
        stream.synchronize()
        pair = []
        for w8, s8, rows, cols in ((wk, sk, H * K, D), (wv, sv, H * D, K)):
            h = C.c_void_p()
            dev._check(L_.tq_qweight_from_device_arrays(dev._ctx, tb.I8_ROW, P(s8), P(w8), rows, cols, C.byref(h)))
            pair.append(h)
        q8.append(pair)
    for B in (1, 16, 64):
        n = max(2, min(16, 128 // B))                  # distinct caches per pass
        cache = rand(n, B, ctx, K + R)
        q, ql, qf, o = rand(H, B, D + R), rand(H, B, K), rand(B, H, K + R), torch.empty((H, B, K), dtype=torch.bfloat16, device="cuda")
        rp, cr, lens = ints(np.full(B, ctx - 1)), ints(np.arange(B) * ctx + ctx - 1), ints(np.full(B, ctx))
        byt, flops = B * ctx * (K + R) * 2, 2.0 * B * ctx * H * (2 * K + R)
        us = graph_ms(lambda: [dev._check(L_.tq_latent_decode(dev._ctx, H, D, R, K, 0.07, R, P(freq), 1.0, 1, P(ql), P(q), D + R, P(cache[i]), B * ctx, P(rp), P(cr), B, ctx,
                                                              P(o))) for i in range(n)]) / n * 1e3
        kernel("decode latent attention", B, us, byt, flops)
        us = graph_ms(lambda: [dev._check(L_.tq_mla_decode(dev._ctx, P(qf), P(cache[i]), P(lens), B, H, K, R, ctx * (K + R), ctx, 0.07, P(o))) for i in range(n)]) / n * 1e3
        kernel("decode latent attention (int8 family)", B, us, byt, flops)
        chunk = 8 if B <= 8 else (B + 15) // 16 * 16
        jobs = ints([(h, h * B + i, min(chunk, B - i), 0) for h in range(H) for i in range(0, B, chunk)])
        nj, o2 = ints([jobs.n // 4]), torch.empty((H * B, K), dtype=torch.bfloat16, device="cuda")
        for what, hs, x, cols, rows in (("absorb W_uk", uk, q, D, K), ("absorb W_uv", uv, ql, K, D)):
            ldx = D + R if what == "absorb W_uk" else K
            us = graph_ms(lambda: [dev._check(L_.tq_dlinear_grouped(dev._ctx, h, P(x), ldx, H * B, P(jobs), P(nj), jobs.n // 4, chunk, rows, null, null, 0.0, 0.0, P(o2),
                                                                    tb.BF16, rows)) for h in hs]) / len(hs) * 1e3
            kernel(what, B, us, H * K * D * 2 + H * B * (K + D) * 2, 2.0 * H * B * K * D)
        qn, qp, y = rand(B, H, D), rand(B, H, R), torch.empty((B, H, K + R), dtype=torch.bfloat16, device="cuda")
        us = graph_ms(lambda: [dev._check(L_.tq_mla_absorb_q(dev._ctx, p[0], P(qn), P(qp), B, H, D, P(y))) for p in q8]) / len(q8) * 1e3
        kernel("absorb W_uk (int8 family)", B, us, H * K * D + H * B * (K + D) * 2, 2.0 * H * B * K * D)
        us = graph_ms(lambda: [dev._check(L_.tq_mla_unabsorb(dev._ctx, p[1], P(o2), B, H, D, P(y), tb.BF16)) for p in q8]) / len(q8) * 1e3
        kernel("absorb W_uv (int8 family)", B, us, H * K * D + H * B * (K + D) * 2, 2.0 * H * B * K * D)
        del cache
        st = [rand(B, lh, ld, lv, dt=tb.F32) for _ in range(max(4, min(64, 128 // B)))]
        x, a1, o = rand(B, width), rand(B, 16, dt=tb.F32), torch.empty((B, lh * lv), dtype=torch.bfloat16, device="cuda")
        us = graph_ms(lambda: [dev._check(lightning(x, t, o, B, B, null, rp, cr, 1)) for t in st]) / len(st) * 1e3
        kernel("decode lightning", B, us, B * lh * ld * lv * 4 * 2)
        us = graph_ms(lambda: [dev._check(recurrence(x, a1, t, o, B, B, null, rp, cr, 1)) for t in st]) / len(st) * 1e3
        kernel("decode gated recurrence", B, us, B * lh * ld * lv * 4 * 2)
        del st
        torch.cuda.empty_cache()

    # ---- prompts
    w_kv = handle(H * 2 * D, K)
    for T in (512, 2048):
        x, a1, st = rand(T, width), rand(T, 16, dt=tb.F32), rand(1, lh, ld, lv, dt=tb.F32)
        cu, rp, o = ints([0, T]), ints(np.arange(T)), torch.empty((T, lh * lv), dtype=torch.bfloat16, device="cuda")
        byt, flops = T * (width + lh * lv) * 2, 2.0 * T * lh * (32 * (ld + lv) + 2 * ld * lv)
        kernel("prefill lightning", T, graph_ms(lambda: dev._check(lightning(x, st, o, T, 1, P(cu), rp, rp, T))) * 1e3, byt, flops)
        kernel("prefill gated recurrence", T, graph_ms(lambda: dev._check(recurrence(x, a1, st, o, T, 1, P(cu), rp, rp, T))) * 1e3, byt, flops)
        sinks = rand(H, dt=tb.F32)
        for name, G, dk, dv, w, sk in (("prefill attention, expanded latents", H, D + R, D, ctx, null), ("prefill attention, all keys (grouped)", 8, D, D, ctx, null),
                                       ("prefill attention, window and sinks", 8, D, D, window, P(sinks)), ("prefill attention, window", 8, D, D, window, null)):
            q, k, v, o = rand(T, H * dk), rand(T, G * dk), rand(T, G * dv), torch.empty((T, H * dv), dtype=torch.bfloat16, device="cuda")
            a = Win(H, G, dk, dv, w, dk ** -0.5, 0.0, float("-inf"))
            us = graph_ms(lambda: dev._check(L_.tq_window_attention_sinks(dev._ctx, C.byref(a), sk, tb.BF16, P(q), H * dk, null, 0, P(k), P(v), T, P(cu), P(rp), P(rp), 1, T, T, T,
                                                                          P(o), H * dv))) * 1e3
            kernel(name, T, us, 0, 2.0 * H * (dk + dv) * sum(min(i + 1, w) for i in range(T)))
        x, y, chunk = rand(T, K), torch.empty((T, H * 2 * D), dtype=torch.bfloat16, device="cuda"), min(T, 256)
        jobs = ints([(0, i, min(chunk, T - i), 0) for i in range(0, T, chunk)])
        nj = ints([jobs.n // 4])
        us = graph_ms(lambda: dev._check(L_.tq_dlinear_grouped(dev._ctx, w_kv, P(x), K, T, P(jobs), P(nj), jobs.n // 4, chunk, H * 2 * D, null, null, 0.0, 0.0, P(y), tb.BF16,
                                                               H * 2 * D))) * 1e3
        kernel("expansion of latents", T, us, (H * 2 * D + T) * K * 2 + T * H * 2 * D * 2, 2.0 * T * K * H * 2 * D)
        us = graph_ms(lambda: dev._check(L_.tq_dlinear(dev._ctx, w_kv, P(x), K, T, P(y), tb.BF16, H * 2 * D))) * 1e3
        kernel("linear of the same size", T, us, (H * 2 * D + T) * K * 2 + T * H * 2 * D * 2, 2.0 * T * K * H * 2 * D)

    # ---- row operators
    G, D, n = 8, 128, 20
    for m in (1, 64, 2048):
        for S in (2, 4):
            xs = [rand(m, S, 4096, dt=tb.F32) for _ in range(n if m < 2048 else 4)]
            y, gain, h = rand(m * 3, 4096, dt=tb.F32), rand(4096, dt=tb.F32), torch.empty((m, 4096), dtype=torch.bfloat16, device="cuda")
            mix, co, slots, wt = rand(S, S, std=0.3, dt=tb.F32), rand(S, dt=tb.F32), ints(np.random.permutation(3 * m)), rand(m, 3, dt=tb.F32)
            us = graph_ms(lambda: [dev._check(L_.tq_stream_mix(dev._ctx, S, S, P(x), P(x), P(y), null, null, 1, null, null, P(mix), P(co), P(co), P(gain), m, 4096, 1e-6, P(h),
                                                               tb.BF16, 4096, null)) for x in xs]) / len(xs) * 1e3
            kernel(f"{S} streams, next norm", m, us, m * 4096 * (8 * S + 6))
            us = graph_ms(lambda: [dev._check(L_.tq_stream_mix(dev._ctx, S, S, P(x), P(x), P(y), P(slots), P(wt), 3, P(h), P(y), P(mix), P(co), P(co), P(gain), m, 4096, 1e-6,
                                                               P(h), tb.BF16, 4096, null)) for x in xs]) / len(xs) * 1e3
            kernel(f"{S} streams, next norm, three experts and a shared one", m, us, m * 4096 * (8 * S + 2 + 16))
        xs = [rand(m, 4096, dt=tb.F32) for _ in range(n if m < 2048 else 8)]
        us = graph_ms(lambda: [dev._check(L_.tq_add_norm(dev._ctx, P(x), P(y), P(slots), 2, P(gain), P(gain), m, 4096, 1e-6, P(h), tb.BF16, 4096)) for x in xs]) / len(xs) * 1e3
        kernel("post-norm, stream, next norm over two experts", m, us, m * 4096 * 18)
        q, raw, keys, qg, rp, fr = rand(m, H * D), rand(m, G * D), rand(m, G * D), rand(H * D), ints(np.arange(m)), rand(32, dt=tb.F32)
        us = graph_ms(lambda: [dev._check(L_.tq_head_norm_rope(dev._ctx, tb.BF16, H, G, D, P(q), H * D, D, P(raw), P(keys), m, P(qg), P(qg), 0, 64, 0, P(fr), 1.0, 1e-6, P(rp),
                                                               P(rp), m)) for _ in range(n)]) / n * 1e3
        kernel("per-head norm and rotation", m, us, m * (H + G) * D * 4)
        us = graph_ms(lambda: [dev._check(L_.tq_qk_norm_rope(dev._ctx, tb.BF16, H, G, D, P(q), H * D, P(raw), P(keys), m, P(qg), P(qg), 64, P(fr), 1.0, 1e-6, P(rp), P(rp), m))
                               for _ in range(n)]) / n * 1e3
        kernel("whole-projection norm and rotation", m, us, m * (H + G) * D * 4)
        q = rand(H, m, 192)
        us = graph_ms(lambda: [dev._check(L_.tq_head_norm_rope(dev._ctx, tb.BF16, H, 0, 192, P(q), 192, m * 192, null, null, m, null, null, 128, 64, 1, P(fr), 1.0, 1e-6, P(rp),
                                                               P(rp), m)) for _ in range(n)]) / n * 1e3
        kernel("rotation of latent queries", m, us, m * H * 192 * 4)
        z, corr = rand(m, 40, dt=tb.F32), rand(40, std=0.01, dt=tb.F32)
        bufs = [ints(np.zeros(m * 5)) for _ in range(4)] + [ints(np.zeros(4 * (m * 5 + 40))), ints([0])]
        us = graph_ms(lambda: [dev._check(L_.tq_route_rule(dev._ctx, P(z), m, 40, 5, 1, 1, P(corr), 8, 8, *map(P, bufs))) for _ in range(n)]) / n * 1e3
        kernel("corrected routing, 5 of 32 + 8", m, us, m * 40 * 4)
        us = graph_ms(lambda: [dev._check(L_.tq_route(dev._ctx, P(z), m, 40, 5, 0, 0, 8, *map(P, bufs))) for _ in range(n)]) / n * 1e3
        kernel("routing, 5 of 40", m, us, m * 40 * 4)
    out["clocks"] = sampler.stop(t_start, time.perf_counter())
    print(json.dumps(out))


# ----------------------------------------------------------------------------------------------
# --sakinex: the Sakinex family (bf16) beside the Numuzen family at equal width, head sizes, window and active feed-forward,
# random weights: decode and prefill throughput of both, and the new kernels beside the like ones, against their rooflines.
# ----------------------------------------------------------------------------------------------
SAKINEX_SIZES = {
    # `top` experts of ff values and the shared one together are as wide as the other models' feed-forward
    "8b": {**{k: NUMUZEN_SIZES["8b"][k] for k in ("layers", "width", "heads", "kv", "dim", "vocab")}, "state": 2048, "pool": 16, "taps": 4, "experts": 8, "top": 2,
           "ff": 4096, "shared": 6144},
    "1b": {**{k: NUMUZEN_SIZES["1b"][k] for k in ("layers", "width", "heads", "kv", "dim", "vocab")}, "state": 1024, "pool": 16, "taps": 4, "experts": 32, "top": 4,
           "ff": 1536, "shared": 2048},
}


def build_sakinex(dev, tb, torch, stream, s, max_seq, max_batch, window):
    from tang_b200 import sakinex as sx

    gen = torch.Generator(device="cuda").manual_seed(7)
    H, G, D, R, d, taps = s["heads"], s["kv"], s["dim"], s["state"], s["width"], s["taps"]
    layer = sx.SakinexLayer(H, G, D, D, D ** -0.5, R, window, s["pool"], taps, sx.Rotation(64, 500000.0, 4.0, 4096, 32.0, 1.0), 0.7, 1.1,
                            sx.Experts(s["experts"], s["top"], s["ff"], s["shared"]))
    cfg = tb.SakinexConfig(s["vocab"], d, 1e-6, 0.5, taps, [layer] * s["layers"])
    model = tb.SakinexModel(dev, cfg, tb.BF16, max_batch, max_seq)
    shapes = {sx.EMBED: (s["vocab"], d), sx.HEAD: (s["vocab"], d), sx.CANON1: (d, taps), sx.CANON2: (d, taps), sx.Q: (H * D, d), sx.K: (G * D, d), sx.V: (G * D, d),
              sx.Q_CONV: (H * D, taps), sx.K_CONV: (G * D, taps), sx.V_CONV: (G * D, taps), sx.LEFT_O: (d, H * D), sx.Z: (R, d), sx.Z_BIAS: (1, R), sx.X: (R, d),
              sx.X_BIAS: (1, R), sx.G: (R, d), sx.RIGHT_O: (d, R), sx.ROUTER: (s["experts"], d), sx.ROUTER_BIAS: (1, s["experts"]), sx.GATE: (s["ff"], d),
              sx.UP: (s["ff"], d), sx.DOWN: (d, s["ff"]), sx.SHARED_GATE: (s["shared"], d), sx.SHARED_UP: (s["shared"], d), sx.SHARED_DOWN: (d, s["shared"])}
    pool = {}
    for name, tensor, i, e in sx.tensor_names(cfg):
        r, c = shapes.get(tensor, (1, d))
        level = 1.0 if tensor in (sx.NORM1, sx.NORM2, sx.FINAL_NORM) else 0.0
        key = (r, c, level, tensor == sx.ROUTER and i)
        if key not in pool:
            with torch.cuda.stream(stream):
                pool[key] = (torch.randn((r, c), device="cuda", generator=gen) * (0.02 if r == 1 else 0.3 if c == taps else c ** -0.5) + level).bfloat16()
            stream.synchronize()
        model.put_pointer(tensor, i, pool[key].data_ptr(), tb.BF16, r, c, e)
    return model


def run_sakinex(args) -> None:
    import ctypes as C

    import torch

    import tang_b200 as tb

    torch.cuda.set_device(0)
    dev = tb.QuantComputeDevice(0)
    L_ = dev._L
    stream = torch.cuda.ExternalStream(dev.stream, device=torch.device("cuda", 0))
    peaks = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json"))) if os.path.exists(os.path.join(ROOT, "MEASURED_PEAKS.json")) else {}
    hbm, tf = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    ctx, window = 2048, 512
    sampler = ClockSampler(0)
    sampler.start()
    t_start = time.perf_counter()

    def graph_ms(fn, reps=10):
        fn()
        dev.sync()
        dev.begin_capture()
        fn()
        g = dev.end_capture()
        ms = _time_ms(torch, stream, dev, g.launch, reps, warm=3)
        g.free()
        return ms

    def rand(*shape, std=1.0, dt=None):
        with torch.cuda.stream(stream):
            t = torch.randn(shape, device="cuda") * std
            t = t if dt == tb.F32 else t.bfloat16()
        stream.synchronize()
        return t

    P = lambda t: C.c_void_p(t.data_ptr() if hasattr(t, "data_ptr") else t.ptr)
    ints = lambda a: dev.upload(np.asarray(a, np.int32).reshape(-1), tb.I32)
    null = C.c_void_p(0)
    touched = lambda experts, top, rows: experts * (1 - (1 - top / experts) ** rows)      # expected number of experts that `rows` rows choose
    out = {"metric": "sakinex_throughput", "unit": "tokens/s", "data": "synthetic", "dtype": "bf16", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf},
           "window": window, "models": [], "kernels": []}
    batches = [1, 2, 4, 8, 16, 64]

    def time_model(size, name, model, s, decode_bytes, prefill_flops):
        row = {"size": size, "model": name, "decode": {}, "prefill": {}}
        for B in batches:
            tok = ints(np.random.randint(0, s["vocab"], B))
            pos, lg = ints(np.full(B, ctx)), dev.alloc(B * s["vocab"], tb.F32)
            ms = graph_ms(lambda: model.decode(tok, pos, B, ctx + 1, lg))
            row["decode"][B] = {"ms": ms, "tokens_per_s": B / ms * 1e3, "frac_of_hbm": decode_bytes(B) / ms / 1e6 / hbm}
        for T in (512, ctx):
            tok = ints(np.random.randint(0, s["vocab"], T))
            cu, st, last, lg = ints([0, T]), ints([0]), ints([T - 1]), dev.alloc(s["vocab"], tb.F32)
            ms = graph_ms(lambda: model.step(tok, T, cu, st, None, 1, T, T, last, 1, lg), 3)
            row["prefill"][T] = {"ms": ms, "tokens_per_s": T / ms * 1e3, "frac_of_bf16": T * prefill_flops(T) / ms / 1e9 / tf}
        out["models"].append(row)
        model.destroy()
        torch.cuda.empty_cache()

    for size in [x for x in args.sakinex.split(",") if x in SAKINEX_SIZES]:
        s = SAKINEX_SIZES[size]
        d, H, G, D, R = s["width"], s["heads"], s["kv"], s["dim"], s["state"]
        mixers, one = s["layers"] * d * ((2 * H + 2 * G) * D + 4 * R), 3 * d * s["ff"]
        fixed = 2 * (mixers + s["layers"] * d * ((s["experts"] + 1) + 3 * s["shared"]) + s["vocab"] * d)
        seen = window + (ctx - window + 1) // s["pool"]
        per_row = s["layers"] * (G * 2 * D * 2 * seen + R * 8 + (s["taps"] - 1) * 2 * (2 * d + (H + 2 * G) * D) * 2)
        active = mixers + s["layers"] * (s["top"] * one + 3 * d * s["shared"])
        time_model(size, "sakinex", build_sakinex(dev, tb, torch, stream, s, ctx + 1, max(batches), window), s,
                   lambda B: fixed + 2 * s["layers"] * one * touched(s["experts"], s["top"], B) + B * per_row, lambda T: 2.0 * active)
        if not args.sakinex_only:
            z = NUMUZEN_SIZES[size]
            gh, gd, gv = z["gla"]
            zm = z["layers"] // 2 * (d * (3 * H + z["kv"]) * D + d * (2 * gh * gd + 3 * gh * gv + 16))
            zone, zrow = 3 * d * z["ff"], z["layers"] // 2 * (z["kv"] * 2 * D * 2 * window + gh * gd * gv * 8)
            time_model(size, "numuzen", build_numuzen(dev, tb, torch, stream, z, ctx + 1, max(batches), window), z,
                       lambda B: 2 * (zm + z["layers"] * z["experts"] * d + z["vocab"] * d + z["layers"] * zone * touched(z["experts"], z["top"], B)) + B * zrow,
                       lambda T: 2.0 * (zm + z["layers"] * z["top"] * zone))

    def kernel(name, m, us, byt=0.0, flops=0.0):
        roof = max(byt / hbm / 1e3, flops / tf / 1e6)
        out["kernels"].append({"kernel": name, "m": m, "us": round(us, 2), "roofline_us": round(roof, 2), "frac": round(roof / us, 3)})

    class Win(C.Structure):
        _fields_ = [(k, C.c_uint32) for k in ("heads", "kv_heads", "dim", "vdim", "window")] + [(k, C.c_float) for k in ("scale", "softcap", "sink")]

    class Gla(C.Structure):
        _fields_ = [(k, C.c_uint32) for k in ("heads", "dim", "vdim", "rank")] + [(k, C.c_float) for k in ("tau", "q_scale", "eps")]

    class Heads(C.Structure):
        _fields_ = [(n, C.c_uint32) for n in ("heads", "kv_heads", "dim", "vdim", "k0", "v0", "channels", "taps", "rot_dims")] + [("norm", C.c_int)] + [
            (n, C.c_uint32) for n in ("pool", "pool_rows")] + [(n, C.c_float) for n in ("rot_mult", "eps")]

    H, G, D, d, pool, taps = 32, 8, 128, 4096, 16, 4
    prow, span = ctx // pool, (H + 2 * G) * D
    lh, ld, lv, R = 16, 128, 256, 4096
    gw = 2 * lh * ld + 2 * lh * lv
    a2, a2b, gnorm = rand(lh * ld, 16, dt=tb.F32), rand(lh * ld, dt=tb.F32), rand(lv, dt=tb.F32)
    zb, ub, freq, cw = rand(R, dt=tb.F32), rand(R, dt=tb.F32), rand(32, dt=tb.F32), rand(taps, span, std=0.4, dt=tb.F32)
    dw, gain = rand(taps, d, std=0.3, dt=tb.F32), rand(d, dt=tb.F32)

    def attention(pooled, w, q, k, v, pk, pv, o, B, rows, n_seqs, cu, rp, cr, max_q):
        a = Win(H, G, D, D, w, D ** -0.5, 0.0, float("-inf"))
        tail = (cu, P(rp), P(cr), n_seqs, rows, max_q, ctx, P(o), H * D)
        if pooled:
            return L_.tq_window_attention_pooled(dev._ctx, C.byref(a), null, tb.BF16, P(q), H * D, null, 0, P(k), P(v), B * ctx, pool, P(pk), P(pv), prow, ctx, 1.0, *tail)
        return L_.tq_window_attention(dev._ctx, C.byref(a), tb.BF16, P(q), H * D, null, 0, P(k), P(v), B * ctx, *tail)

    def min_gru(x, st, o, rows, n_seqs, cu, rp, cr, max_q):
        off = lambda c: C.c_void_p(x.data_ptr() + 2 * c)
        return L_.tq_min_gru(dev._ctx, tb.BF16, R, off(0), off(R), off(2 * R), 3 * R, P(zb), P(ub), 1.0, P(st), ctx, n_seqs * ctx, cu, P(rp), P(cr), n_seqs, rows, max_q, P(o), R)

    def recurrence(x, a1, st, o, rows, n_seqs, cu, rp, cr, max_q):
        g, off = Gla(lh, ld, lv, 16, 16.0, ld ** -0.5, 1e-6), lambda c: C.c_void_p(x.data_ptr() + 2 * c)
        return L_.tq_gla(dev._ctx, C.byref(g), tb.BF16, off(0), off(lh * ld), off(2 * lh * ld), off(2 * lh * ld + lh * lv), gw, P(a1), 16, P(a2), P(a2b), P(gnorm),
                         P(st), ctx, n_seqs * ctx, cu, P(rp), P(cr), n_seqs, rows, max_q, P(o), lh * lv)

    def heads(x, st, q, k, v, pk, pv, rows, n_seqs, cu, rp, cr, max_q, max_len):
        a = Heads(H, G, D, D, H * D, (H + G) * D, span, taps, 64, 1, pool, prow, 1.1, 1e-6)
        return L_.tq_conv_heads(dev._ctx, C.byref(a), tb.BF16, P(x), span, P(cw), P(st), P(freq), ctx, n_seqs * ctx, cu, P(rp), P(cr), n_seqs, rows, max_q, max_len, P(q),
                                H * D, P(k), P(v), P(pk), P(pv))

    seen = window + (ctx - window) // pool
    one, fac = torch.ones(1, device="cuda"), torch.full((1,), 0.5, device="cuda")
    torch.cuda.synchronize()
    # ---- one row per sequence
    for B in (1, 16, 64):
        n = max(2, min(16, 128 // B))                  # distinct caches per pass
        k, v, pk, pv = rand(n, B, ctx, G * D), rand(n, B, ctx, G * D), rand(n, B, prow, G * D), rand(n, B, prow, G * D)
        q, o = rand(B, H * D), torch.empty((B, H * D), dtype=torch.bfloat16, device="cuda")
        rp, cr = ints(np.full(B, ctx - 1)), ints(np.arange(B) * ctx + ctx - 1)
        for name, pooled, w, rows in (("pooled blocks and window", 1, window, seen), ("window", 0, window, window), ("window of as many keys", 0, seen, seen)):
            us = graph_ms(lambda: [dev._check(attention(pooled, w, q, k[i], v[i], pk[i], pv[i], o, B, B, B, null, rp, cr, 1)) for i in range(n)]) / n * 1e3
            kernel(f"decode attention, {name}", B, us, B * rows * G * D * 2 * 2)
        N = 24
        xs, sts = [rand(B, span) for _ in range(N)], [rand(B, taps - 1, span) for _ in range(N)]
        us = graph_ms(lambda: [dev._check(heads(x, t, q, k[0], v[0], pk[0], pv[0], B, B, null, rp, cr, 1, ctx)) for x, t in zip(xs, sts)]) / N * 1e3
        kernel("convolved heads", B, us, B * span * 2 * (2 + 2 * (taps - 1)))
        rp16 = ints(np.full(B, ctx - pool))
        cr16 = ints(np.arange(B) * ctx + ctx - pool)
        us = graph_ms(lambda: [dev._check(heads(x, t, q, k[0], v[0], pk[0], pv[0], B, B, null, rp16, cr16, 1, ctx)) for x, t in zip(xs, sts)]) / N * 1e3
        kernel("convolved heads, a block is complete", B, us, B * (span * 2 * (2 + 2 * (taps - 1)) + 2 * G * D * 2 * (pool + 1)))
        qg = rand(D)
        us = graph_ms(lambda: [dev._check(L_.tq_head_norm_rope(dev._ctx, tb.BF16, H, G, D, P(x), span, D, P(k[0]), P(v[0]), B * ctx, P(qg), P(qg), 0, 64, 0, P(freq), 1.0, 1e-6,
                                                               P(rp), P(cr), B)) for x in xs]) / N * 1e3
        kernel("per-head norm and rotation", B, us, B * (H + G) * D * 4)
        del k, v, pk, pv
        x, st = rand(B, 3 * R), [rand(B, R, dt=tb.F32) for _ in range(32)]
        o = torch.empty((B, R), dtype=torch.bfloat16, device="cuda")
        us = graph_ms(lambda: [dev._check(min_gru(x, t, o, B, B, null, rp, cr, 1)) for t in st]) / len(st) * 1e3
        kernel("decode minGRU", B, us, B * R * (3 * 2 + 2 + 8))
        st = [rand(B, lh, ld, lv, dt=tb.F32) for _ in range(max(4, min(64, 128 // B)))]
        x, a1, o = rand(B, gw), rand(B, 16, dt=tb.F32), torch.empty((B, lh * lv), dtype=torch.bfloat16, device="cuda")
        us = graph_ms(lambda: [dev._check(recurrence(x, a1, t, o, B, B, null, rp, cr, 1)) for t in st]) / len(st) * 1e3
        kernel("decode gated recurrence", B, us, B * lh * ld * lv * 4 * 2)
        del st
        xs, h = [rand(B, d, dt=tb.F32) for _ in range(N)], torch.empty((B, d), dtype=torch.bfloat16, device="cuda")
        y, slots, wt, cs, gate = rand(2 * B, d, dt=tb.F32), ints(np.random.permutation(2 * B)), rand(B, 2, dt=tb.F32), [rand(B, taps - 1, d) for _ in range(N)], rand(B, dt=tb.F32)
        for name, experts in (("stream, next norm and convolution", 0), ("stream, next norm and convolution over two experts and a gated one", 1)):
            us = graph_ms(lambda: [dev._check(L_.tq_stream_step(dev._ctx, P(x), P(x), P(y), P(slots) if experts else null, P(wt) if experts else null, 2, P(y) if experts else null,
                                                                P(gate) if experts else null, 1, null, P(one), P(fac), P(gain), B, d, 1e-6, P(dw), P(t), taps, ctx, P(rp),
                                                                P(cr), P(h), tb.BF16, d, null)) for x, t in zip(xs, cs)]) / N * 1e3
            kernel(name, B, us, B * d * (14 + 4 * (taps - 1) + 8 * experts))
        for name, r_, n_, byt in (("post-norm, stream, next norm", null, 1, 14), ("post-norm, stream, next norm over two experts", P(slots), 2, 18)):
            us = graph_ms(lambda: [dev._check(L_.tq_add_norm(dev._ctx, P(x), P(y), r_, n_, P(gain), P(gain), B, d, 1e-6, P(h), tb.BF16, d)) for x in xs]) / N * 1e3
            kernel(name, B, us, B * d * byt)
        torch.cuda.empty_cache()

    # ---- prompts
    for T in (512, 2048):
        cu, rp = ints([0, T]), ints(np.arange(T))
        q, k, v, pk, pv = rand(T, H * D), rand(ctx, G * D), rand(ctx, G * D), rand(prow, G * D), rand(prow, G * D)
        o = torch.empty((T, H * D), dtype=torch.bfloat16, device="cuda")
        for w in (128, window):
            for name, pooled in (("pooled blocks and window", 1), ("window", 0)):
                us = graph_ms(lambda: dev._check(attention(pooled, w, q, k, v, pk, pv, o, 1, T, 1, P(cu), rp, rp, T))) * 1e3
                kernel(f"prefill attention, {name} {w}", T, us, 0, 4.0 * H * D * sum(min(i + 1, w) + (max(0, i - w + 1) // pool if pooled else 0) for i in range(T)))
        N = 8 if T == 512 else 4
        xs, st = [rand(T, span) for _ in range(N)], rand(1, taps - 1, span)
        us = graph_ms(lambda: [dev._check(heads(x, st, q, k, v, pk, pv, T, 1, P(cu), rp, rp, T, T)) for x in xs]) / N * 1e3
        kernel("convolved heads, pooled blocks, states (3 kernels)", T, us, T * span * 4)
        qg = rand(D)
        us = graph_ms(lambda: [dev._check(L_.tq_head_norm_rope(dev._ctx, tb.BF16, H, G, D, P(x), span, D, P(k), P(v), ctx, P(qg), P(qg), 0, 64, 0, P(freq), 1.0, 1e-6, P(rp),
                                                               P(rp), T)) for x in xs]) / N * 1e3
        kernel("per-head norm and rotation", T, us, T * (H + G) * D * 4)
        xs, st, o = [rand(T, 3 * R) for _ in range(N)], rand(1, R, dt=tb.F32), torch.empty((T, R), dtype=torch.bfloat16, device="cuda")
        us = graph_ms(lambda: [dev._check(min_gru(x, st, o, T, 1, P(cu), rp, rp, T)) for x in xs]) / N * 1e3
        kernel("prefill minGRU", T, us, T * R * 8)
        x, a1, st = rand(T, gw), rand(T, 16, dt=tb.F32), rand(1, lh, ld, lv, dt=tb.F32)
        us = graph_ms(lambda: dev._check(recurrence(x, a1, st, o, T, 1, P(cu), rp, rp, T))) * 1e3
        kernel("prefill gated recurrence", T, us, T * (gw + lh * lv) * 2, 2.0 * T * lh * (32 * (ld + lv) + 2 * ld * lv))
        xs, st, h = [rand(T, d) for _ in range(2 * N)], rand(1, taps - 1, d), torch.empty((T, d), dtype=torch.bfloat16, device="cuda")
        us = graph_ms(lambda: [dev._check(L_.tq_conv_residual(dev._ctx, tb.BF16, d, taps, P(dw), P(st), ctx, ctx, P(x), d, P(cu), P(rp), P(rp), 1, T, T, T, P(h), d))
                               for x in xs]) / len(xs) * 1e3
        kernel("input convolution, states (2 kernels)", T, us, T * d * 4)
        xs = [rand(T, d, dt=tb.F32) for _ in range(N)]
        us = graph_ms(lambda: [dev._check(L_.tq_rms_norm(dev._ctx, P(x), tb.F32, null, P(gain), tb.F32, T, d, 1e-6, P(h), tb.BF16, null)) for x in xs]) / N * 1e3
        kernel("plain norm", T, us, T * d * 6)
        y, slots, wt, gate = rand(2 * T, d, dt=tb.F32), ints(np.random.permutation(2 * T)), rand(T, 2, dt=tb.F32), rand(T, dt=tb.F32)
        us = graph_ms(lambda: [dev._check(L_.tq_stream_step(dev._ctx, P(x), P(x), P(y), P(slots), P(wt), 2, P(y), P(gate), 1, null, P(one), P(fac), P(gain), T, d, 1e-6, null, null,
                                                            0, 1, P(rp), P(rp), P(h), tb.BF16, d, null)) for x in xs]) / N * 1e3
        kernel("stream, next norm over two experts and a gated one", T, us, T * d * 22)
        us = graph_ms(lambda: [dev._check(L_.tq_add_norm(dev._ctx, P(x), P(y), P(slots), 2, P(gain), P(gain), T, d, 1e-6, P(h), tb.BF16, d)) for x in xs]) / N * 1e3
        kernel("post-norm, stream, next norm over two experts", T, us, T * d * 18)
    for m in (1, 64, 2048):
        z, bias = rand(m, 33, dt=tb.F32), rand(32, std=0.1, dt=tb.F32)
        bufs = [ints(np.zeros(m * 4)) for _ in range(4)] + [ints(np.zeros(4 * (m * 4 + 32))), ints([0])]
        us = graph_ms(lambda: [dev._check(L_.tq_route_biased(dev._ctx, P(z), 33, m, 32, 4, 1, 1, P(bias), null, 0, 8, *map(P, bufs))) for _ in range(20)]) / 20 * 1e3
        kernel("biased routing, 4 of 32", m, us, m * 33 * 4)
        us = graph_ms(lambda: [dev._check(L_.tq_route(dev._ctx, P(z), m, 32, 4, 0, 0, 8, *map(P, bufs))) for _ in range(20)]) / 20 * 1e3
        kernel("routing, 4 of 32", m, us, m * 32 * 4)
    out["clocks"] = sampler.stop(t_start, time.perf_counter())
    print(json.dumps(out))


def main() -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=50)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--m", type=int, default=1, help="decode tokens per GEMV (1..64)")
    ap.add_argument("--layers", type=int, default=32, help="distinct weight matrices per step")
    ap.add_argument("--cpu-budget", type=float, default=8.0, help="seconds of CPU baseline timing")
    ap.add_argument("--ref-sample", type=int, default=4, help="matvecs per step of the reference arm")
    ap.add_argument("--no-cpu-baseline", action="store_true")
    ap.add_argument("--no-decode", action="store_true", help="skip the Llama-3-8B-shaped decode step")
    ap.add_argument("--no-extras", action="store_true", help="skip the M sweep / MoE / MLA timings (N=1 only)")
    ap.add_argument("--decode-batches", default="1,16,64")
    ap.add_argument("--decode-layers", type=int, default=32)
    ap.add_argument("--decode-steps", type=int, default=10)
    ap.add_argument("--tofazen", nargs="?", const="8b,1b", default="", help="time the Tofazen family instead (sizes: 8b, 1b, or none: kernels only)")
    ap.add_argument("--tofazen-only", action="store_true", help="with --tofazen: leave the int4 model out")
    ap.add_argument("--numuzen", nargs="?", const="8b,1b", default="", help="time the Numuzen family instead (sizes: 8b, 1b, or none: kernels only)")
    ap.add_argument("--dotanex", nargs="?", const="8b,1b", default="", help="time the Dotanex family instead (sizes: 8b, 1b, or none: kernels only)")
    ap.add_argument("--dotanex-only", action="store_true", help="with --dotanex: leave the Numuzen model out")
    ap.add_argument("--sakinex", nargs="?", const="8b,1b", default="", help="time the Sakinex family instead (sizes: 8b, 1b, or none: kernels only)")
    ap.add_argument("--sakinex-only", action="store_true", help="with --sakinex: leave the Numuzen model out")
    ap.add_argument("--numuzen-only", action="store_true", help="with --numuzen: leave the Tofazen model out")
    args = ap.parse_args()
    if args.sakinex:
        run_sakinex(args)
        return
    if args.dotanex:
        run_dotanex(args)
        return
    if args.numuzen:
        run_numuzen(args)
        return
    if args.tofazen:
        run_tofazen(args)
        return
    args.warmup = max(args.warmup, 3) if args.impl == "ours" else args.warmup
    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if args.impl == "reference":
        run_reference(args, rank)
        return
    if world != args.gpus and world == 1 and args.gpus > 1:
        sys.exit("--gpus N > 1 must be launched with torch.distributed.run (one rank per GPU)")
    run_ours(args, rank, world, local_rank)


if __name__ == "__main__":
    main()
