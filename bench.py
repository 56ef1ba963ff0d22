#!/usr/bin/env python
"""Benchmark of the fused grouped-query-attention hot path.

  python bench.py [--gpus N] [--steps K] [--warmup W] [--impl ours|reference]
                  [--workload prefill|decode]

One JSON line on stdout (rank 0).  A step is one pass of the hot path over one
batch of synthetic input:
  prefill (default, the headline): BASELINE config 2 — bf16, batch 8, seq 2048,
      32 query / 4 KV heads, head_dim 64, causal, RoPE fused.  Metric: attention
      TFLOP/s with the algorithmic count 4*B*Hq*S^2*D/2.
  decode: BASELINE config 3 — batch 64, paged bf16 KV cache (16-token pages),
      lengths uniform in [1024, 4096].  Metric: HBM GB/s over the algorithmic
      bytes 1024 * sum(L_i).  The prefill line also carries a `decode` object
      with this measurement.
With N > 1 (torchrun, one rank per GPU) every rank processes its own copy of
the workload (weak scaling, no data-path collective); the time is the max over
ranks.  `--impl reference` times the reference's OWN CUDA operators (its
attention-layer core, through oracle/_ref, host arrays in and out) when that
library was built, and the plain-C restatement of its operators on the host
cores beside it (the reference has no CPU implementation of this path: its
operators throw "only GPU implementation available").
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import tempfile
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

_emit = print

PREFILL = dict(B=8, S=2048, Hq=32, Hkv=4, D=64)
DECODE = dict(B=64, Hq=32, Hkv=4, D=64, Lmin=1024, Lmax=4096, page=16)


def _ncu_traffic():
    """dram__bytes_read.sum + dram__bytes_write.sum per launch, from the ncu captures summarised under profiles/
    (profiles/ncu_dram_traffic.json holds the figures of those summaries)."""
    try:
        d = json.load(open(os.path.join(ROOT, "profiles", "ncu_dram_traffic.json")))
        return {k: float(v["read"]) + float(v["write"]) for k, v in d.items() if isinstance(v, dict)}
    except Exception:
        return {}


class _Traffic(dict):
    def __missing__(self, key):
        return None


NCU_TRAFFIC = _Traffic(_ncu_traffic())


# nominal figures, beside the measured ones the fractions are taken against: dense bf16 2250 TFLOP/s, HBM3e 8000 GB/s
NOMINAL_TENSOR_TFLOPS = 2250.0
NOMINAL_HBM_GBS = 8000.0


def peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        d = json.load(open(p))
        return dict(hbm=float(d["hbm_gbs"]), tensor=float(d["bf16_tflops"]), source="measured")
    return dict(hbm=6650.0, tensor=1590.0, source="fallback")


def prefill_flops(c=PREFILL):
    return 4.0 * c["B"] * c["Hq"] * c["S"] * c["S"] * c["D"] / 2.0


# ----------------------------------------------------------------------------- clocks
class ClockSampler:
    FIELDS = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
              "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
              "clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int):
        self.index, self.proc, self.path = index, None, None

    def start(self):
        try:
            fd, self.path = tempfile.mkstemp(suffix=".csv")
            os.close(fd)
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", str(self.index), f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits",
                 "-lms", "100"], stdout=open(self.path, "w"), stderr=subprocess.DEVNULL)
        except Exception:
            self.proc = None

    def stop(self):
        out = {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        if self.proc is None:
            return out
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except Exception:
            self.proc.kill()
        rows = []
        for line in open(self.path):
            parts = [x.strip() for x in line.split(",")]
            if len(parts) >= 7:
                try:
                    rows.append((float(parts[0]), float(parts[1]), float(parts[2]), parts[3:7]))
                except ValueError:
                    pass
        os.unlink(self.path)
        if not rows:
            return out
        # "under load" = samples drawing the most power
        pw = sorted(r[2] for r in rows)
        thr = pw[len(pw) // 2]
        load = [r for r in rows if r[2] >= thr] or rows
        sm = sorted(r[0] for r in load)
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = sorted({names[i] for r in rows for i in range(4) if r[3][i].lower().startswith("active")})
        out.update(sm_mhz=sm[len(sm) // 2], sm_max_mhz=rows[0][1], reasons=reasons, samples=len(rows),
                   power_w_max=max(r[2] for r in rows))
        return out


# ----------------------------------------------------------------------------- CPU arm
def cpu_prefill_sample(n_batches: int, steps: int = 1, warmup: int = 0):
    """Times the plain-C restatement (all host threads) on `n_batches` batch elements of config 2."""
    import numpy as np
    from oracle import cref, ref_attention as R
    # all the host cores this process may use (torchrun presets OMP_NUM_THREADS=1 for its children)
    cref.set_num_threads(len(os.sched_getaffinity(0)))
    c = PREFILL
    rng = np.random.default_rng(0)
    q = R.round_bf16(rng.standard_normal((n_batches, c["S"], c["Hq"], c["D"]), dtype=np.float32))
    k = R.round_bf16(rng.standard_normal((n_batches, c["S"], c["Hkv"], c["D"]), dtype=np.float32))
    v = R.round_bf16(rng.standard_normal((n_batches, c["S"], c["Hkv"], c["D"]), dtype=np.float32))
    for _ in range(warmup):
        cref.attention_per_head(q, k, v, causal=True, round_bf16=True, batches=(0, 1), heads=(0, 2))
    t0 = time.perf_counter()
    for _ in range(steps):
        cref.attention_per_head(q, k, v, causal=True, round_bf16=True)
    dt = (time.perf_counter() - t0) / steps
    flops = prefill_flops() * n_batches / c["B"]
    return dict(value=flops / dt / 1e12, seconds=dt, cores=cref.num_threads(),
                sample=f"{n_batches} of {c['B']} batch elements of config 2 (all 32 heads, S=2048), "
                       f"oracle/ref_attention.c with OpenMP")


def reference_cuda_sample(n_batches: int, steps: int, warmup: int):
    """Times the reference's OWN CUDA operators (oracle/_ref, compiled from the reference tree): per batch element
    the operator sequence of its attention layer core -- op_rope on q and k, host-side head repeat, op_mm, op_multiply,
    causal op_softmax, op_mm -- on fp32 host arrays, as its tensors require (upload and download are part of its call).
    None when that library or a GPU is not there."""
    import numpy as np
    from oracle import cref
    try:
        import torch
        if not torch.cuda.is_available() or not os.path.exists(cref._GPU_SO):
            return None
        cref.gpu()
    except Exception:
        return None
    c = PREFILL
    rng = np.random.default_rng(0)
    q = rng.standard_normal((n_batches, c["S"], c["Hq"] * c["D"]), dtype=np.float32)
    k = rng.standard_normal((n_batches, c["S"], c["Hkv"] * c["D"]), dtype=np.float32)
    v = rng.standard_normal((n_batches, c["S"], c["Hkv"] * c["D"]), dtype=np.float32)

    def one_step():
        for b in range(n_batches):
            cref.gpu_attention_core(q[b], k[b], v[b], num_heads=c["Hq"], num_kv_heads=c["Hkv"], head_dim=c["D"],
                                    causal=True)

    for _ in range(warmup):
        one_step()
    t0 = time.perf_counter()
    for _ in range(steps):
        one_step()
    dt = (time.perf_counter() - t0) / steps
    flops = prefill_flops() * n_batches / c["B"]
    return dict(value=flops / dt / 1e12, seconds=dt,
                sample=f"{n_batches} of {c['B']} batch elements of config 2 (S=2048, 32q/4kv, D=64), the reference's own "
                       f"CUDA operators (fp32, heads collapsed as its layer computes them) via oracle/_ref, host arrays in "
                       f"and out")


def run_reference_arm(args):
    """The reference's own implementation of the path.  The reference has no CPU implementation of it (its
    operators throw "only GPU implementation available"), so what can be timed of its OWN code is its CUDA
    operators, through oracle/_ref: that is this arm's value whenever that library and a GPU are present, and it
    says so (`reference_class`).  Because that code runs on a GPU, under torchrun EVERY rank runs it on its own GPU
    (the same per-GPU sample; value = all ranks' work / the slowest rank's time), so that a ratio against the other
    arm at N GPUs compares N GPUs with N GPUs.  The plain-C restatement on the host cores is timed beside it on rank
    0 alone (`cpu_port`); without oracle/_ref it is the arm's value and only rank 0 works."""
    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    n_batches = 2
    ref_steps, ref_warmup = max(1, min(args.steps, 5)), (1 if args.warmup else 0)
    gpu = None
    try:
        import torch
        if torch.cuda.is_available():
            torch.cuda.set_device(local)
            gpu = reference_cuda_sample(n_batches=n_batches, steps=ref_steps, warmup=ref_warmup)
    except Exception:
        gpu = None
    ranks_that_ran = 1
    if world > 1:
        import torch
        import torch.distributed as dist
        dist.init_process_group("gloo")
        t = torch.tensor([gpu["seconds"] if gpu is not None else -1.0], dtype=torch.float64)
        lo = t.clone()
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        dist.all_reduce(lo, op=dist.ReduceOp.MIN)
        if gpu is not None and float(lo.item()) > 0:      # every rank has timed its GPU
            gpu = dict(gpu, seconds=float(t.item()), value=gpu["value"] * gpu["seconds"] / float(t.item()) * world)
            ranks_that_ran = world
        elif gpu is not None:
            gpu = None if rank != 0 else gpu
        dist.destroy_process_group()
    if rank != 0:
        return
    cpu_steps = max(1, min(args.steps, 3))
    cpu = cpu_prefill_sample(n_batches=n_batches, steps=cpu_steps, warmup=1 if args.warmup else 0)
    r = gpu if gpu is not None else cpu
    steps_run, warmup_run = (ref_steps, ref_warmup) if gpu is not None else (cpu_steps, 1 if args.warmup else 0)
    line = {
        "impl": "reference", "metric": "prefill_attention_tflops", "value": r["value"], "unit": "TFLOP/s",
        "n_gpus": args.gpus, "steps": steps_run, "warmup": warmup_run,
        "steps_requested": args.steps, "warmup_requested": args.warmup,
        "ms_per_step": r["seconds"] * 1e3,
        "ms_per_step_note": f"one step = {n_batches} of the {PREFILL['B']} batch elements of config 2 per GPU; value is "
                            f"scaled to the metric's unit (FLOP of the sample / its time), not to the full batch time",
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "f32", "data": "synthetic",
        "reference_class": ("the reference's own CUDA operators on the GPU (fp32 SIMT, heads collapsed as its layer "
                            "computes them); the reference has no CPU implementation of this path") if gpu is not None
                           else "plain-C restatement of the reference's operators on the host cores",
        "config": {"workload": "prefill attention core, BASELINE config 2 (B=8 S=2048 32q/4kv D=64 causal, RoPE fused)",
                   "sample": r["sample"], "ranks_that_ran": ranks_that_ran},
        "cpu_baseline": {"value": r["value"], "unit": "TFLOP/s", "cores": 0 if gpu is not None else cpu["cores"],
                         "kind": "reference" if gpu is not None else "port",
                         "device": "gpu: reference CUDA ops (no CPU path exists)" if gpu is not None else "host cores",
                         "sample": r["sample"]},
        "cpu_port": {"value": cpu["value"], "unit": "TFLOP/s", "cores": cpu["cores"], "kind": "port",
                     "sample": cpu["sample"], "steps": cpu_steps},
        "e2e": {"value": r["value"], "unit": "TFLOP/s", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
        "gpu_launches": 0,
    }
    _emit(json.dumps(line))


# ----------------------------------------------------------------------------- GPU arm
def make_decode_case(torch, seed, n_sets):
    import numpy as np
    from baranet_bdml_b200.kv_cache import PagedKVCache
    c = DECODE
    rng = np.random.default_rng(seed)
    lens = rng.integers(c["Lmin"], c["Lmax"] + 1, c["B"])
    pages = (lens + c["page"] - 1) // c["page"]
    n_pages = int(pages.sum())
    max_pages = c["Lmax"] // c["page"]
    caches = []
    for s in range(n_sets):
        cache = PagedKVCache(n_pages, c["B"], max_pages, c["Hkv"], c["D"])
        cache.pool.copy_(torch.randn(cache.pool.shape, device="cuda", dtype=torch.float32).to(torch.bfloat16))
        perm = rng.permutation(n_pages).astype(np.int32)
        pt = np.zeros((c["B"], max_pages), dtype=np.int32)
        at = 0
        for b in range(c["B"]):
            pt[b, :pages[b]] = perm[at:at + pages[b]]
            at += pages[b]
        cache.page_table.copy_(torch.from_numpy(pt))
        cache.seq_lens.copy_(torch.from_numpy(lens.astype(np.int32)))
        caches.append(cache)
    q = torch.randn((c["B"], c["Hq"], c["D"]), device="cuda").to(torch.bfloat16)
    bytes_alg = int(lens.sum()) * c["Hkv"] * c["D"] * 2 * 2
    return caches, q, bytes_alg, int(lens.sum())


def time_loop(torch, fn, steps, warmup, dist=None):
    """W untimed + K timed calls of fn(i); CUDA events on the current stream, barrier + sync on both sides."""
    for i in range(warmup):
        fn(i)
    torch.cuda.synchronize()
    if dist is not None:
        dist.barrier()
        torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for i in range(steps):
        fn(warmup + i)
    e1.record()
    torch.cuda.synchronize()
    if dist is not None:
        dist.barrier()
    return e0.elapsed_time(e1) / steps   # ms per step


def measure_prefill(torch, ops, args, rank, world, dist, reduce_max, pk):
    c = PREFILL
    B, S, Hq, Hkv, D = c["B"], c["S"], c["Hq"], c["Hkv"], c["D"]
    # rotate over 3 input sets (3 x 151 MB > 126 MB L2)
    n_sets = 3
    g = torch.Generator(device="cuda").manual_seed(1234 + rank)
    sets = []
    for _ in range(n_sets):
        q = torch.randn((B, S, Hq, D), generator=g, device="cuda").to(torch.bfloat16)
        k = torch.randn((B, S, Hkv, D), generator=g, device="cuda").to(torch.bfloat16)
        v = torch.randn((B, S, Hkv, D), generator=g, device="cuda").to(torch.bfloat16)
        o = torch.empty_like(q)
        sets.append((q, k, v, o, ops.prefill_workspace(B, S, Hq, Hkv, D)))

    def step(i):
        q, k, v, o, ws = sets[i % n_sets]
        ops.attn_prefill_bf16(q, k, v, out=o, workspace=ws)

    def kernel_only(i):
        q, k, v, o, ws = sets[i % n_sets]
        ops.attn_prefill_bf16(q, k, v, out=o, workspace=ws, reuse_rotated_k=True)

    ms_step = reduce_max(time_loop(torch, step, args.steps, args.warmup, dist))
    ms_kernel = time_loop(torch, kernel_only, args.steps, max(3, args.warmup))   # attention kernel alone
    for s in sets:
        s[4].status()

    # end to end: pinned host buffers, H2D + kernels + D2H inside the timed region
    ms_e2e, h2d, d2h = None, 0, 0
    if not args.no_e2e:
        hq = torch.randn((B, S, Hq, D)).to(torch.bfloat16).pin_memory()
        hk = torch.randn((B, S, Hkv, D)).to(torch.bfloat16).pin_memory()
        hv = torch.randn((B, S, Hkv, D)).to(torch.bfloat16).pin_memory()
        ho = torch.empty((B, S, Hq, D), dtype=torch.bfloat16).pin_memory()
        # the public host-memory front-end: per step the H2D copy of that step's q/k/v, both kernels and the D2H copy
        # of its output, on three streams over two device buffer sets (copies of neighbouring steps overlap)
        pipe = ops.HostPrefillPipeline(B, S, Hq, Hkv, D, depth=2)
        hos = [ho, torch.empty_like(ho).pin_memory()]

        def e2e_loop(steps):
            for i in range(steps):
                pipe.submit(hq, hk, hv, hos[i % 2])
            pipe.finish()

        e2e_loop(max(3, args.warmup))
        torch.cuda.synchronize()
        if dist is not None:
            dist.barrier()
            torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        e2e_loop(args.steps)
        e1.record()            # after finish(): the current stream has waited for the last D2H copy
        torch.cuda.synchronize()
        if dist is not None:
            dist.barrier()
        pipe.status()
        ms_e2e = reduce_max(e0.elapsed_time(e1) / args.steps)
        h2d = (hq.numel() + hk.numel() + hv.numel()) * 2
        d2h = ho.numel() * 2
        # the floor of that number: the same bytes moved by plain copies with no kernel at all (H2D of q, k, v on one
        # stream, D2H of an output-sized buffer on another, every rank at once) - one cudaMemcpyAsync per tensor
        dq, dk, dv, do_ = (torch.empty_like(t, device="cuda") for t in (hq, hk, hv, ho))
        s_in, s_out = torch.cuda.Stream(), torch.cuda.Stream()

        def copies(steps):
            for _ in range(steps):
                with torch.cuda.stream(s_in):
                    dq.copy_(hq, non_blocking=True)
                    dk.copy_(hk, non_blocking=True)
                    dv.copy_(hv, non_blocking=True)
                with torch.cuda.stream(s_out):
                    ho.copy_(do_, non_blocking=True)
            torch.cuda.current_stream().wait_stream(s_in)
            torch.cuda.current_stream().wait_stream(s_out)

        copies(3)
        torch.cuda.synchronize()
        if dist is not None:
            dist.barrier()
            torch.cuda.synchronize()
        c0, c1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        s_in.wait_stream(torch.cuda.current_stream())
        s_out.wait_stream(torch.cuda.current_stream())
        c0.record()
        s_in.wait_stream(torch.cuda.current_stream())
        s_out.wait_stream(torch.cuda.current_stream())
        copies(args.steps)
        c1.record()
        torch.cuda.synchronize()
        if dist is not None:
            dist.barrier()
        ms_copies = reduce_max(c0.elapsed_time(c1) / args.steps)
        del dq, dk, dv, do_

    flops = prefill_flops()
    ach = flops / (ms_kernel * 1e-3) / 1e12
    sharded = None
    if world > 1 and B % world == 0:
        # The partition BASELINE config 2 states: its 8 x 4 (batch, KV-head group) units dealt batch-major to the
        # ranks, no collective (strong scaling: at 8 GPUs one batch element = 4 units each).
        Bs = B // world
        sh = [(q[:Bs].contiguous(), k[:Bs].contiguous(), v[:Bs].contiguous(), torch.empty_like(q[:Bs]),
               ops.prefill_workspace(Bs, S, Hq, Hkv, D)) for (q, k, v, _, _) in sets]

        def sstep(i):
            q, k, v, o, ws = sh[i % n_sets]
            ops.attn_prefill_bf16(q, k, v, out=o, workspace=ws)

        ms_own = time_loop(torch, sstep, args.steps, args.warmup, dist)
        ms_sh = reduce_max(ms_own)
        sharded = {"scaling": "strong", "value": flops / (ms_sh * 1e-3) / 1e12, "unit": "TFLOP/s", "ms_per_step": ms_sh,
                   "ms_per_step_by_rank": _all_ranks(torch, dist, ms_own), "units_per_rank": Bs * Hkv,
                   "workload": f"ONE config-2 batch (8 sequences, 32 (batch, KV-group) units) over {world} ranks, "
                               f"{Bs} batch element(s) = {Bs * Hkv} units each; time = slowest rank"}
        del sh
    result_extra = {"sharded": sharded} if sharded is not None else {}
    return {
        **result_extra,
        "metric": "prefill_attention_tflops", "value": flops * world / (ms_step * 1e-3) / 1e12, "unit": "TFLOP/s",
        "n_gpus": world, "steps": args.steps, "warmup": args.warmup, "ms_per_step": ms_step,
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {"workload": "prefill attention core, BASELINE config 2: bf16 in / fp32 accumulate, per GPU batch 8, "
                               "seq 2048, 32 query / 4 KV heads, head_dim 64, causal, RoPE theta 1e4 fused, "
                               "positions 0..2047",
                   "global_batch": B * world, "seq_len": S, "parallelism": f"batch-sharded x{world}, no collective",
                   "l2": f"inputs rotate over {n_sets} buffer sets of 151 MB each (> 126 MB L2)",
                   "flops_per_step_per_gpu": flops, "launches_per_step": 2},
        "roofline": {"bound": "tensor", "achieved": ach, "peak": pk["tensor"], "unit": "TFLOP/s",
                     "frac": ach / pk["tensor"], "traffic": NCU_TRAFFIC["prefill_kernel"],
                     "traffic_unit": "bytes of DRAM traffic per launch (ncu capture, profiles/prefill_kernel_config2.md)",
                     "peak_source": pk["source"] + " (bf16 burst)",
                     "frac_of_nominal": ach / NOMINAL_TENSOR_TFLOPS, "nominal_peak": NOMINAL_TENSOR_TFLOPS,
                     "kernel": "prefill_kernel", "kernel_ms": ms_kernel},
        "e2e": None if ms_e2e is None else {
            "value": flops * world / (ms_e2e * 1e-3) / 1e12, "unit": "TFLOP/s", "h2d_bytes_per_step": h2d,
            "d2h_bytes_per_step": d2h, "ms_per_step": ms_e2e,
            "copies_only_ms_per_step": ms_copies, "fraction_of_copies_only": ms_copies / ms_e2e,
            "copies_only_note": "the same H2D + D2H bytes per step as plain concurrent copies on every rank, no kernel: "
                                "the floor that the host links set for this number",
            "api": "ops.HostPrefillPipeline.submit per step (pinned host q/k/v/out; H2D, kernels and D2H of "
                   "neighbouring steps overlap on three streams over two device buffer sets)"},
        "gpu_launches": 2 * args.steps,
    }


def _all_ranks(torch, dist, x):
    """x (float) of every rank, as a list (rank order)."""
    if dist is None:
        return [x]
    t = torch.tensor([x], device="cuda", dtype=torch.float64)
    out = [torch.zeros_like(t) for _ in range(dist.get_world_size())]
    dist.all_gather(out, t)
    return [float(o.item()) for o in out]


def make_decode_shard(torch, lens_all, mine, seed, n_sets):
    """Caches holding the sequences `mine` (indices into lens_all) of one decode batch."""
    import numpy as np
    from baranet_bdml_b200.kv_cache import PagedKVCache
    c = DECODE
    rng = np.random.default_rng(seed)
    lens = np.asarray([lens_all[i] for i in mine], dtype=np.int64)
    pages = (lens + c["page"] - 1) // c["page"]
    n_pages, max_pages, nb = int(pages.sum()), c["Lmax"] // c["page"], len(mine)
    caches = []
    for _ in range(n_sets):
        cache = PagedKVCache(max(n_pages, 1), nb, max_pages, c["Hkv"], c["D"])
        cache.pool.copy_(torch.randn(cache.pool.shape, device="cuda", dtype=torch.float32).to(torch.bfloat16))
        perm = rng.permutation(max(n_pages, 1)).astype(np.int32)
        pt = np.zeros((nb, max_pages), dtype=np.int32)
        at = 0
        for b in range(nb):
            pt[b, :pages[b]] = perm[at:at + pages[b]]
            at += pages[b]
        cache.page_table.copy_(torch.from_numpy(pt))
        cache.seq_lens.copy_(torch.from_numpy(lens.astype(np.int32)))
        caches.append(cache)
    q = torch.randn((nb, c["Hq"], c["D"]), device="cuda").to(torch.bfloat16)
    return caches, q, int(lens.sum())


def measure_decode(torch, args, rank, world, dist, reduce_max, pk):
    dsets = 8   # 8 x ~168 MB of cache: every launch reads HBM-cold data
    caches, q, bytes_alg, tokens = make_decode_case(torch, 77 + rank, dsets)
    outs = torch.empty((DECODE["B"], DECODE["Hq"], DECODE["D"]), dtype=torch.bfloat16, device="cuda")

    def dstep(i):
        caches[i % dsets].decode(q, num_heads=DECODE["Hq"], out=outs, max_seq_len=DECODE["Lmax"], rope_q=True)

    dsteps = args.steps if args.decode_only else max(args.steps, 16)
    ms_own = time_loop(torch, dstep, dsteps, max(3, args.warmup), dist)
    ms_dec = reduce_max(ms_own)
    per_rank = _all_ranks(torch, dist, ms_own)
    per_rank_bytes = _all_ranks(torch, dist, float(bytes_alg))
    # the same launches replayed from a CUDA graph (what a serving loop does; no host work between the launches)
    ms_graph = None
    try:
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            for i in range(dsets):
                dstep(i)
        torch.cuda.current_stream().wait_stream(side)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            for i in range(dsets):
                dstep(i)
        ms_graph = reduce_max(time_loop(torch, lambda i: graph.replay(), max(4, dsteps // dsets), 3, dist)) / dsets
        del graph
    except Exception as e:
        ms_graph = None
    for cch in caches:
        cch.status()
    ms_eager = ms_dec
    if ms_graph:
        ms_dec = ms_graph        # the launches replayed from a CUDA graph: no host work between them
    gbs = bytes_alg / (ms_dec * 1e-3) / 1e9
    out = {
        "metric": "decode_attention_hbm_gbs", "value": sum(per_rank_bytes) / (ms_dec * 1e-3) / 1e9, "unit": "GB/s",
        "ms_per_step": ms_dec, "ms_per_step_eager": ms_eager,
        "timing": ("8 launches (one per rotating cache) replayed from a CUDA graph, CUDA events around the replays; "
                   "ms_per_step_eager is the same launches issued one by one from Python") if ms_graph else
                  "launches issued one by one, CUDA events around them",
        "steps": dsteps, "n_gpus": world, "scaling": "weak",
        "config": {"workload": "paged decode, BASELINE config 3: per GPU batch 64, one token per sequence, bf16 "
                               "KV cache in 16-token pages (permuted page table), lengths uniform in [1024,4096]",
                   "tokens_in_cache": tokens, "algorithmic_bytes_per_step": bytes_alg,
                   "l2": f"{dsets} distinct caches rotate"},
        "roofline": {"bound": "hbm", "achieved": gbs, "peak": pk["hbm"], "unit": "GB/s", "frac": gbs / pk["hbm"],
                     "traffic": NCU_TRAFFIC["decode_paged_kernel"],
                     "traffic_unit": "bytes of DRAM traffic per launch (ncu capture, profiles/decode_paged_kernel_config3.md)",
                     "peak_source": pk["source"], "frac_of_nominal": gbs / NOMINAL_HBM_GBS,
                     "nominal_peak": NOMINAL_HBM_GBS, "kernel": "decode_paged_kernel"},
        "ms_per_step_eager_by_rank": per_rank,
        "gpu_launches": dsteps,
    }
    del caches
    torch.cuda.empty_cache()
    if world > 1:
        # The partition BASELINE config 3 states: ONE batch of 64 sequences, every rank the sequences that a
        # longest-first greedy assignment by length gives it (strong scaling: the work per GPU shrinks with N, so
        # the launch is latency-bound at 8 GPUs: about 20 MB per GPU against a fixed start-up and tail).
        import numpy as np
        from baranet_bdml_b200 import dist as bdist
        lens_all = np.random.default_rng(77).integers(DECODE["Lmin"], DECODE["Lmax"] + 1, DECODE["B"])
        mine = bdist.shard_sequences_by_length(lens_all, world)[rank]
        sh_caches, sh_q, sh_tokens = make_decode_shard(torch, lens_all, mine, 1000 + rank, dsets)
        sh_out = torch.empty((len(mine), DECODE["Hq"], DECODE["D"]), dtype=torch.bfloat16, device="cuda")

        def sstep(i):
            sh_caches[i % dsets].decode(sh_q, num_heads=DECODE["Hq"], out=sh_out, max_seq_len=DECODE["Lmax"], rope_q=True)

        ms_sh_own = time_loop(torch, sstep, dsteps, max(3, args.warmup), dist)
        ms_sh = reduce_max(ms_sh_own)
        total_bytes = int(lens_all.sum()) * DECODE["Hkv"] * DECODE["D"] * 4
        out["sharded"] = {
            "scaling": "strong", "value": total_bytes / (ms_sh * 1e-3) / 1e9, "unit": "GB/s", "ms_per_step": ms_sh,
            "ms_per_step_by_rank": _all_ranks(torch, dist, ms_sh_own),
            "tokens_by_rank": [int(x) for x in _all_ranks(torch, dist, float(sh_tokens))],
            "sequences_by_rank": [int(x) for x in _all_ranks(torch, dist, float(len(mine)))],
            "workload": "the SAME 64 sequences of config 3 sharded over the ranks by length (greedy, longest first), "
                        "no collective; time = slowest rank",
            "algorithmic_bytes_per_step": total_bytes}
        for cch in sh_caches:
            cch.status()
        del sh_caches
        torch.cuda.empty_cache()
    return out


def measure_rmsnorm(torch, args, rank, world, dist, reduce_max, pk):
    """Row N3 (the step either side of attention): residual add + RMSNorm over the tokens of config 2
    (16384 rows x hidden 2048, fp32 like the reference).  One launch reads a and b and writes the sum and the normed
    rows: 4 x 134 MB = 537 MB per step, every byte once; larger than L2, so no buffer rotation is needed."""
    from baranet_bdml_b200 import _lib
    rows, hidden = PREFILL["B"] * PREFILL["S"], 2048
    g = torch.Generator(device="cuda").manual_seed(99 + rank)
    a = torch.randn((rows, hidden), generator=g, device="cuda")
    b = torch.randn((rows, hidden), generator=g, device="cuda")
    w = torch.ones((hidden,), device="cuda")
    s_out, y = torch.empty_like(a), torch.empty_like(a)
    L = _lib.load()

    def fused(i):
        _lib.check(L.bn_add_rmsnorm_f32(a.data_ptr(), hidden, 1, b.data_ptr(), hidden, 1, w.data_ptr(), 1,
                                        s_out.data_ptr(), hidden, 1, y.data_ptr(), hidden, 1, rows, hidden, 1e-6,
                                        torch.cuda.current_stream().cuda_stream))

    def plain(i):
        _lib.check(L.bn_rmsnorm_f32(a.data_ptr(), hidden, 1, w.data_ptr(), 1, y.data_ptr(), hidden, 1, rows, hidden,
                                    1e-6, torch.cuda.current_stream().cuda_stream))

    steps = max(20, args.steps // 2)
    ms_fused = reduce_max(time_loop(torch, fused, steps, 3, dist))
    ms_plain = reduce_max(time_loop(torch, plain, steps, 3, dist))
    bytes_fused, bytes_plain = 4 * rows * hidden * 4, 2 * rows * hidden * 4
    gbs = bytes_fused * world / (ms_fused * 1e-3) / 1e9
    out = {
        "metric": "add_rmsnorm_hbm_gbs", "value": gbs, "unit": "GB/s", "ms_per_step": ms_fused, "steps": steps,
        "n_gpus": world, "dtype": "f32",
        "config": {"workload": "residual add + RMSNorm (row N3), 16384 rows x hidden 2048 fp32 = the tokens of "
                               "BASELINE config 2; one launch, bit-identical to the reference's op_add + op_rmsnorm",
                   "algorithmic_bytes_per_step": bytes_fused, "l2": "537 MB per step, larger than L2"},
        "roofline": {"bound": "hbm", "achieved": gbs / world, "peak": pk["hbm"], "unit": "GB/s",
                     "frac": gbs / world / pk["hbm"], "traffic": NCU_TRAFFIC["rmsnorm_kernel"],
                     "traffic_unit": "bytes of DRAM traffic per launch (ncu capture, profiles/rmsnorm_kernel_16384x2048.md)",
                     "peak_source": pk["source"], "kernel": "rmsnorm_regs_kernel"},
        "rmsnorm_only": {"value": bytes_plain * world / (ms_plain * 1e-3) / 1e9, "unit": "GB/s",
                         "ms_per_step": ms_plain, "algorithmic_bytes_per_step": bytes_plain},
        "gpu_launches": 2 * steps,
    }
    if rank == 0 and world == 1 and not args.no_cpu_baseline:
        import numpy as np
        from oracle import cref
        cref.set_num_threads(len(os.sched_getaffinity(0)))
        n = 2048
        rng = np.random.default_rng(0)
        xa, xb = rng.standard_normal((n, hidden), dtype=np.float32), rng.standard_normal((n, hidden), dtype=np.float32)
        ww = np.ones(hidden, np.float32)
        cref.add_rmsnorm(xa[:64], xb[:64], ww)
        t0 = time.perf_counter()
        reps = 5
        for _ in range(reps):
            cref.add_rmsnorm(xa, xb, ww)
        dt = (time.perf_counter() - t0) / reps
        out["cpu_baseline"] = {"value": 4 * n * hidden * 4 / dt / 1e9, "unit": "GB/s", "cores": cref.num_threads(),
                               "kind": "port", "sample": f"{n} of {rows} rows, oracle/ref_attention.c with OpenMP"}
    return out


def measure_embed_argmax(torch, args, rank, world, dist, reduce_max, pk):
    """Row N2: greedy argmax over a prefill's logits (2048 rows x 32000, 262 MB read) and the embedding gather of
    config 2's 16384 tokens (134 MB read + 134 MB written), both on the device."""
    from baranet_bdml_b200 import _lib
    L = _lib.load()
    rows, vocab, hidden, n_tok = PREFILL["S"], 32000, 2048, PREFILL["B"] * PREFILL["S"]
    g = torch.Generator(device="cuda").manual_seed(5 + rank)
    logits = torch.randn((rows, vocab), generator=g, device="cuda")
    idx = torch.zeros((rows,), dtype=torch.int32, device="cuda")
    table = torch.randn((vocab, hidden), generator=g, device="cuda")
    ids = torch.randint(0, vocab, (n_tok,), generator=g, device="cuda", dtype=torch.int32)
    emb = torch.empty((n_tok, hidden), device="cuda")

    def amax(i):
        _lib.check(L.bn_argmax_rows_f32(logits.data_ptr(), vocab, 1, idx.data_ptr(), rows, vocab,
                                        torch.cuda.current_stream().cuda_stream))

    def gather(i):
        _lib.check(L.bn_embedding_gather_f32(table.data_ptr(), hidden, ids.data_ptr(), emb.data_ptr(), hidden, n_tok,
                                             hidden, vocab, None, torch.cuda.current_stream().cuda_stream))

    steps = max(20, args.steps // 2)
    ms_a = reduce_max(time_loop(torch, amax, steps, 3, dist))
    ms_g = reduce_max(time_loop(torch, gather, steps, 3, dist))
    b_a, b_g = rows * vocab * 4, 2 * n_tok * hidden * 4
    gbs = b_a * world / (ms_a * 1e-3) / 1e9
    return {
        "metric": "argmax_hbm_gbs", "value": gbs, "unit": "GB/s", "ms_per_step": ms_a, "steps": steps, "n_gpus": world,
        "dtype": "f32",
        "config": {"workload": "per-row argmax of 2048 x 32000 fp32 logits (row N2), first maximum as op_argmax",
                   "algorithmic_bytes_per_step": b_a, "l2": "262 MB per step, larger than L2"},
        "roofline": {"bound": "hbm", "achieved": gbs / world, "peak": pk["hbm"], "unit": "GB/s",
                     "frac": gbs / world / pk["hbm"], "traffic": NCU_TRAFFIC["argmax_rows_kernel"],
                     "traffic_unit": "bytes of DRAM traffic per launch (ncu capture, "
                                     "profiles/argmax_and_embedding_gather_kernels.md)",
                     "peak_source": pk["source"], "kernel": "argmax_rows_kernel"},
        "embedding_gather": {"value": b_g * world / (ms_g * 1e-3) / 1e9, "unit": "GB/s", "ms_per_step": ms_g,
                             "algorithmic_bytes_per_step": b_g,
                             "workload": "16384 token rows of 2048 fp32 from a 32000-row table"},
        "gpu_launches": 2 * steps,
    }


def measure_gemm(torch, ops, args, rank, world, dist, reduce_max, pk):
    """Row N1: the q_proj / o_proj GEMM of the layer at the token count of config 2: (16384, 2048) @ (2048, 2048)^T,
    bf16 operands, fp32 accumulation.  Inputs rotate over 3 activation buffers (3 x 67 MB + weights > L2)."""
    M, N, K = PREFILL["B"] * PREFILL["S"], 2048, 2048
    g = torch.Generator(device="cuda").manual_seed(7 + rank)
    xs = [torch.randn((M, K), generator=g, device="cuda").to(torch.bfloat16) for _ in range(3)]
    w = (torch.randn((N, K), generator=g, device="cuda") * 0.02).to(torch.bfloat16)
    out = torch.empty((M, N), dtype=torch.bfloat16, device="cuda")
    err = torch.zeros(1, dtype=torch.int32, device="cuda")

    def step(i):
        ops.gemm_bf16_nt(xs[i % 3], w, out=out, error_word=err)

    steps = max(20, args.steps // 2)
    ms = reduce_max(time_loop(torch, step, steps, 3, dist))
    if int(err.item()) != 0:
        raise RuntimeError("gemm: a bounded device-side wait ran out")
    flops = 2.0 * M * N * K
    tf = flops * world / (ms * 1e-3) / 1e12
    return {
        "metric": "projection_gemm_tflops", "value": tf, "unit": "TFLOP/s", "ms_per_step": ms, "steps": steps,
        "n_gpus": world, "dtype": "bf16",
        "config": {"workload": "q_proj / o_proj GEMM of the layer (row N1): (16384, 2048) @ (2048, 2048)^T, bf16 in, "
                               "fp32 accumulate, bf16 out", "flops_per_step_per_gpu": flops,
                   "l2": "activations rotate over 3 buffers of 67 MB"},
        "roofline": {"bound": "tensor", "achieved": tf / world, "peak": pk["tensor"], "unit": "TFLOP/s",
                     "frac": tf / world / pk["tensor"], "traffic": NCU_TRAFFIC["gemm_bf16_nt_kernel"],
                     "traffic_unit": "bytes of DRAM traffic per launch (ncu capture, "
                                     "profiles/gemm_bf16_nt_kernel_16384x2048x2048.md)",
                     "peak_source": pk["source"] + " (bf16 burst)", "kernel": "gemm_bf16_nt_kernel"},
        "gpu_launches": steps,
    }


def measure_mlp(torch, ops, args, rank, world, dist, reduce_max, pk):
    """Row N4: the SwiGLU MLP of TinyLLaMA at config 2's token count: fused gate/up GEMM with the SiLU * mul epilogue
    (16384 x 2048 -> 5632, 756 GFLOP) and the down GEMM (5632 -> 2048, 378 GFLOP), two launches."""
    M, K, I = PREFILL["B"] * PREFILL["S"], 2048, 5632
    g = torch.Generator(device="cuda").manual_seed(17 + rank)
    xs = [torch.randn((M, K), generator=g, device="cuda").to(torch.bfloat16) for _ in range(2)]
    wg = (torch.randn((I, K), generator=g, device="cuda") * 0.02).to(torch.bfloat16)
    wu = (torch.randn((I, K), generator=g, device="cuda") * 0.02).to(torch.bfloat16)
    wd = (torch.randn((K, I), generator=g, device="cuda") * 0.02).to(torch.bfloat16)
    gu = ops.pack_gate_up(wg, wu)
    h = torch.empty((M, I), dtype=torch.bfloat16, device="cuda")
    y = torch.empty((M, K), dtype=torch.bfloat16, device="cuda")
    err = torch.zeros(1, dtype=torch.int32, device="cuda")

    def step(i):
        ops.gemm_swiglu_bf16_nt(xs[i % 2], gu, I, out=h, error_word=err)
        ops.gemm_bf16_nt(h, wd, out=y, error_word=err)

    steps = max(10, args.steps // 5)
    ms = reduce_max(time_loop(torch, step, steps, 3, dist))
    if int(err.item()) != 0:
        raise RuntimeError("mlp: a bounded device-side wait ran out")
    flops = 2.0 * M * K * (2 * I) + 2.0 * M * I * K
    tf = flops * world / (ms * 1e-3) / 1e12
    return {
        "metric": "swiglu_mlp_tflops", "value": tf, "unit": "TFLOP/s", "ms_per_step": ms, "steps": steps,
        "n_gpus": world, "dtype": "bf16",
        "config": {"workload": "SwiGLU MLP (row N4): 16384 tokens, hidden 2048, intermediate 5632; fused gate/up GEMM "
                               "with SiLU*mul epilogue + down GEMM", "flops_per_step_per_gpu": flops},
        "roofline": {"bound": "tensor", "achieved": tf / world, "peak": pk["tensor"], "unit": "TFLOP/s",
                     "frac": tf / world / pk["tensor"], "traffic": None,
                     "peak_source": pk["source"] + " (bf16 burst)", "kernel": "gemm_bf16_nt_kernel"},
        "gpu_launches": 2 * steps,
    }


def measure_decoder_layer(torch, args, rank, world, dist, reduce_max, pk):
    """One TinyLLaMA decoder block (hidden 2048, 32q/4kv heads, intermediate 5632) on the bf16 path over config 2's
    tokens (B=8, S=2048): norm, fused q/k/v GEMM (K rotation in its epilogue), fused attention, o GEMM, add+norm, fused
    gate/up GEMM, down GEMM = 7 kernel launches (`layers.LLaMADecoderLayerBF16.forward_parts`)."""
    from baranet_bdml_b200.layers import LLaMAConfig, LLaMADecoderLayerBF16
    import numpy as np
    np.random.seed(1 + rank)
    cfg = LLaMAConfig()
    layer = LLaMADecoderLayerBF16(cfg)
    B, S, H = PREFILL["B"], PREFILL["S"], cfg.hidden_size
    g = torch.Generator(device="cuda").manual_seed(3 + rank)
    xs = [torch.randn((B, S, H), generator=g, device="cuda").to(torch.bfloat16) for _ in range(2)]

    def step(i):
        layer.forward_parts(xs[i % 2])

    steps = max(10, args.steps // 10)
    ms = reduce_max(time_loop(torch, step, steps, 3, dist))
    # the same ten launches replayed from one CUDA graph
    ms_graph = None
    try:
        from baranet_bdml_b200.layers import GraphedDecoderLayerBF16
        graphed = GraphedDecoderLayerBF16(layer, xs[0])
        ms_graph = reduce_max(time_loop(torch, lambda i: graphed.graph.replay(), steps, 3, dist))
    except Exception as e:      # the eager number stands
        ms_graph = repr(e)
    T, I, kv = B * S, cfg.intermediate_size, cfg.num_key_value_heads * cfg.head_dim
    flops = prefill_flops() + 2.0 * T * H * (2 * H + 2 * kv) + 2.0 * T * H * 3 * I
    tf = flops * world / (ms * 1e-3) / 1e12
    return {
        "metric": "decoder_layer_tflops", "value": tf, "unit": "TFLOP/s", "ms_per_step": ms, "steps": steps,
        "n_gpus": world, "dtype": "bf16", "tokens_per_s": T * world / (ms * 1e-3), "ms_per_step_cuda_graph": ms_graph,
        "config": {"workload": "one TinyLLaMA decoder block, bf16, 16384 tokens (B=8, S=2048), causal, 7 kernel launches",
                   "flops_per_step_per_gpu": flops},
        "roofline": {"bound": "tensor", "achieved": tf / world, "peak": pk["tensor"], "unit": "TFLOP/s",
                     "frac": tf / world / pk["tensor"], "traffic": None, "peak_source": pk["source"] + " (bf16 burst)",
                     "kernel": "gemm_bf16_nt_kernel + prefill_kernel"},
        "gpu_launches": 7 * steps,
    }


def measure_longctx(torch, args, rank, world, dist, reduce_max, pk):
    """batch 4, one 262144-token sequence each, 32q/4kv heads.  The sequence is cut into
    contiguous page-aligned token ranges, one per GPU; each GPU decodes over its range (normalised partial
    output + log-sum-exp), the partials are exchanged with ONE all-gather and merged locally."""
    import numpy as np
    from baranet_bdml_b200 import dist as bdist
    from baranet_bdml_b200.kv_cache import PagedKVCache
    B, L, Hq, Hkv, D = 4, 262144, 32, 4, 64
    t0, t1 = bdist.sequence_split_ranges(L, world)[rank]
    Lloc = t1 - t0
    n_pages = B * (Lloc // 16)
    cache = PagedKVCache(n_pages, B, Lloc // 16, Hkv, D)
    cache.pool.copy_(torch.randn(cache.pool.shape, device="cuda", dtype=torch.float32).to(torch.bfloat16))
    rng = np.random.default_rng(5 + rank)
    cache.page_table.copy_(torch.from_numpy(rng.permutation(n_pages).astype(np.int32).reshape(B, Lloc // 16)))
    cache.seq_lens.fill_(Lloc)
    q = torch.randn((B, Hq, D), device="cuda").to(torch.bfloat16)
    qpos = torch.full((B,), L - 1, dtype=torch.int32, device="cuda")
    ex = bdist.PartialExchange(B * Hq, D, mode="peer" if world > 1 else "nccl")
    ex_nccl = bdist.PartialExchange(B * Hq, D) if world > 1 else None
    o32, lse = ex.out_view.view(B, Hq, D), ex.lse_view.view(B, Hq)

    def decode_only(i):
        cache.decode(q, num_heads=Hq, out_f32=o32, lse=lse, q_positions=qpos, max_seq_len=Lloc)

    def exchange_only(i):
        ex.combine()

    def exchange_nccl_only(i):
        ex_nccl.combine()

    def step(i):
        decode_only(i)
        if world > 1:
            ex.combine()

    # ---- checks before any timing (bench values of a wrong result are worth nothing)
    # (1) this rank's partial for (sequence 0, query head 0) over ALL its tokens against plain fp32 arithmetic
    step(0)
    torch.cuda.synchronize()
    pt0 = cache.page_table[0].long()
    kv = cache.pool[pt0, 0].float()                              # (pages, K|V, 16, D) of KV head 0
    K0, V0 = kv[:, 0].reshape(-1, D), kv[:, 1].reshape(-1, D)
    i2 = torch.arange(D // 2, device="cuda", dtype=torch.float32)
    freq = (1.0 / torch.pow(torch.tensor(10000.0, device="cuda"), 2.0 * i2 / D)).float()
    ang = float(L - 1) * freq
    qf = q[0, 0].float()
    qr = torch.empty_like(qf)
    qr[0::2] = qf[0::2] * torch.cos(ang) - qf[1::2] * torch.sin(ang)
    qr[1::2] = qf[0::2] * torch.sin(ang) + qf[1::2] * torch.cos(ang)
    sc = (K0 @ qr) * 0.125
    ref_lse = torch.logsumexp(sc, 0)
    ref_out = torch.softmax(sc, 0) @ V0
    err_partial = max(float((o32[0, 0] - ref_out).abs().max()), float((lse[0, 0] - ref_lse).abs()))
    # (2) the merged result against the log-sum-exp merge written out in fp64 on the gathered partials, and
    #     identical on every rank
    err_merge, rank_diff = 0.0, 0.0
    if world > 1:
        ex_nccl.send.copy_(ex.send)
        ex_nccl.combine()
        torch.cuda.synchronize()
        ex.status()
        allp = ex_nccl.recv.view(world, -1)
        outs = allp[:, : B * Hq * D].reshape(world, B * Hq, D).double()
        lses = allp[:, B * Hq * D:].reshape(world, B * Hq).double()
        m = lses.max(0).values
        wgt = torch.exp(lses - m)
        ref_merged = (wgt[:, :, None] * outs).sum(0) / wgt.sum(0)[:, None]
        err_merge = float((ex.out.double() - ref_merged).abs().max())
        mine = ex.out.clone()
        dist.broadcast(mine, 0)
        rank_diff = float((mine - ex.out).abs().max())
    checks = {"max_abs_err_partial_vs_fp32": reduce_max(err_partial), "max_abs_err_merge_vs_fp64": reduce_max(err_merge),
              "max_abs_diff_between_ranks": reduce_max(rank_diff)}
    if checks["max_abs_err_partial_vs_fp32"] > 2e-2 or checks["max_abs_err_merge_vs_fp64"] > 1e-3 or checks["max_abs_diff_between_ranks"] != 0.0:
        raise RuntimeError(f"long-context decode check failed: {checks}")
    del kv, K0, V0, sc

    steps = max(args.steps // 4, 8)
    ms_eager = reduce_max(time_loop(torch, step, steps, 3, dist))
    # the same steps replayed from a CUDA graph, 8 steps per replay: two launches per step issued from Python cost the
    # host more than the step costs the GPU once the shard is small (the exchange keeps its step number in its
    # buffer, so a captured launch can be replayed)
    ms, timing = ms_eager, "launches issued one by one from Python"
    if world > 1 and ex._peer is not None:
        per_graph = 8
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.stream(side):
            with torch.cuda.graph(graph, stream=side):
                for i in range(per_graph):
                    step(i)
        torch.cuda.current_stream().wait_stream(side)
        ms = reduce_max(time_loop(torch, lambda i: graph.replay(), max(steps // per_graph, 4), 2, dist)) / per_graph
        timing = f"{per_graph} steps (decode kernel + exchange) per CUDA-graph replay; ms_per_step_eager is the same issued one by one from Python"
        torch.cuda.synchronize()
        ex.status()
        # the replayed steps still merge correctly: the result of the last one against the eager one (same inputs)
        eager_out = ex.out.clone()
        step(0)
        torch.cuda.synchronize()
        if not torch.equal(eager_out, ex.out):
            raise RuntimeError("long-context decode: graph-replayed step differs from the eager step")
    ms_dec_own = time_loop(torch, decode_only, steps, 3, dist)
    ms_dec = reduce_max(ms_dec_own)
    ms_ex = reduce_max(time_loop(torch, exchange_only, steps * 4, 3, dist)) if world > 1 else 0.0
    ms_ex_nccl = reduce_max(time_loop(torch, exchange_nccl_only, steps * 4, 3, dist)) if world > 1 else 0.0
    cache.status()
    ex.status()
    bytes_alg = B * L * Hkv * D * 2 * 2           # the whole job, all ranks
    gbs = bytes_alg / (ms * 1e-3) / 1e9
    return {
        "metric": "long_context_decode_hbm_gbs", "value": gbs, "unit": "GB/s", "ms_per_step": ms,
        "ms_per_step_eager": ms_eager, "timing": timing, "steps": steps, "n_gpus": world, "scaling": "strong",
        "config": {"workload": "split-KV decode, BASELINE config 4: batch 4, KV length 262144 bf16 (1 GiB of cache in "
                               "total), 32q/4kv heads, sequence split across the GPUs, partials merged by one "
                               "exchange + log-sum-exp combine",
                   "algorithmic_bytes_per_step": bytes_alg, "tokens_per_gpu": Lloc, "exchange": ex.kind,
                   "l2": "cache per GPU is %d MiB" % (B * Lloc * Hkv * D * 4 >> 20)},
        "roofline": {"bound": "hbm", "achieved": gbs / world, "peak": pk["hbm"], "unit": "GB/s",
                     "frac": gbs / world / pk["hbm"], "traffic": None, "peak_source": pk["source"],
                     "frac_of_nominal": gbs / world / NOMINAL_HBM_GBS, "nominal_peak": NOMINAL_HBM_GBS,
                     "kernel": "decode_paged_kernel", "note": "per GPU; includes the exchange when n_gpus > 1"},
        "step_split_ms": {"decode_kernel": ms_dec, "decode_kernel_by_rank": _all_ranks(torch, dist, ms_dec_own),
                          "exchange_and_merge": ms_ex, "exchange_and_merge_nccl_all_gather": ms_ex_nccl,
                          "note": "each part timed alone, back to back; the step runs them in sequence"},
        "checks": checks,
        "gpu_launches": steps * (1 if world == 1 else 2),   # + the exchange per step when n_gpus > 1
    }


def measure_generate(torch, args, rank, world, dist, reduce_max, pk):
    """TinyLLaMA-1.1B generation on the new kernels, random weights N(0, 0.02): 22 layers, hidden
    2048, SwiGLU 5632, vocab 32000, 32q/4kv heads; 16 prompts of 512 ids uniform in [0, 32000), then 128 greedy decode
    steps (prompt pass filling the paged caches, then one row per sequence per token, the step replayed from a CUDA
    graph).  With N GPUs the 16 prompts are dealt to the ranks (2 each at 8), weights replicated, no collective."""
    from baranet_bdml_b200 import layers as L
    from baranet_bdml_b200.model import LLaMAModelBF16
    import numpy as np
    n_prompts, S, new_tokens = 16, 512, int(getattr(args, "generate_steps", 128) or 128)
    if n_prompts % world:
        return {"error": f"16 prompts do not divide over {world} ranks"}
    B = n_prompts // world
    cfg = L.LLaMAConfig()
    cfg.rms_norm_eps = 1e-5                      # BASELINE config 5; the reference's own default is 1e-6
    np.random.seed(11)
    with L.device_init(0.02, seed=100):          # same weights on every rank (replicas)
        model = LLaMAModelBF16(cfg)
    g = torch.Generator(device="cuda").manual_seed(500 + rank)
    ids = torch.randint(0, cfg.vocab_size, (B, S), generator=g, device="cuda", dtype=torch.int32)

    def run_once():
        e = [torch.cuda.Event(enable_timing=True) for _ in range(3)]
        e[0].record()
        logits = model.prefill(ids, S + new_tokens)
        nxt = model.argmax(logits)
        e[1].record()
        step = model.capture_decode_step()      # capture is outside the decode timing below
        torch.cuda.synchronize()
        e2 = [torch.cuda.Event(enable_timing=True) for _ in range(2)]
        e2[0].record()
        tok = nxt
        for _ in range(new_tokens):
            _, tok = step(tok)
        e2[1].record()
        torch.cuda.synchronize()
        return e[0].elapsed_time(e[1]), e2[0].elapsed_time(e2[1]), tok.clone()

    run_once()                                   # warm-up: workspaces, kernel attributes, graph capture paths
    if dist is not None:
        dist.barrier()
    # three whole generations, the median of each part (the eager prompt pass follows the host's load)
    runs = [run_once()[:2] for _ in range(1 if args.generate_only else 3)]
    ms_prefill = sorted(r[0] for r in runs)[len(runs) // 2]
    ms_decode = sorted(r[1] for r in runs)[len(runs) // 2]
    ms_prefill, ms_decode = reduce_max(ms_prefill), reduce_max(ms_decode)
    model.status()
    n_params = sum(int(t.numel()) for t in model.parameters())
    total_ms = ms_prefill + ms_decode
    out = {
        "metric": "generate_tokens_per_s", "value": n_prompts * new_tokens / (ms_decode * 1e-3), "unit": "tokens/s",
        "n_gpus": world, "scaling": "strong" if world > 1 else "weak", "dtype": "bf16",
        "prefill_ms": ms_prefill, "prefill_tokens_per_s": n_prompts * S / (ms_prefill * 1e-3),
        "decode_ms_per_step": ms_decode / new_tokens, "decode_steps": new_tokens,
        "end_to_end_ms": total_ms, "end_to_end_new_tokens_per_s": n_prompts * new_tokens / (total_ms * 1e-3),
        "config": {"workload": "BASELINE config 5: TinyLLaMA-1.1B, 22 layers, hidden 2048, intermediate 5632, vocab 32000, "
                               "32q/4kv heads, head_dim 64; 16 prompts x 512 ids, 128 greedy decode steps; weights "
                               "N(0, 0.02); bf16 weights and activations, fp32 accumulation",
                   "prompts_per_gpu": B, "parameters": n_params, "rms_norm_eps": 1e-5,
                   "rms_norm_eps_note": "BASELINE config 5 says 1e-5; the reference's LLaMAConfig default is 1e-6",
                   "parallelism": f"prompts dealt to {world} rank(s), weights replicated, no collective",
                   "decode": "one CUDA-graph replay per token (7 launches per block + 4 of this library, and 6 small "
                             f"torch kernels: casts, the length vector); prompt pass eager; median of {len(runs)} generation(s)"},
        "gpu_launches": len(runs) * (new_tokens * (7 * cfg.num_hidden_layers + 4) + 7 * cfg.num_hidden_layers + 5),
    }
    del model
    torch.cuda.empty_cache()
    return out


def measure_layer_f32(torch, args, rank, world, pk):
    """BASELINE config 1 through the drop-in fp32 layer (S=128, hidden 2048, 32q/4kv heads, collapsed-head
    semantics, the reference's result to 1e-5) next to the reference's own operator sequence for the same layer on
    the same GPU (oracle/_ref, when that library is there)."""
    import numpy as np
    from baranet_bdml_b200.layers import GroupedQueryAttention, LLaMAConfig
    from baranet_bdml_b200.tensor import AGTensor
    rng = np.random.default_rng(0)
    cfg = LLaMAConfig()
    x = rng.standard_normal((128, 2048)).astype(np.float32)
    w = {k: (rng.standard_normal(shape) * 0.02).astype(np.float32)
         for k, shape in (("q", (2048, 2048)), ("k", (2048, 256)), ("v", (2048, 256)), ("o", (2048, 2048)))}
    attn = GroupedQueryAttention(cfg, is_cuda=True)
    attn.q_proj, attn.k_proj = AGTensor(w["q"], is_cuda=True), AGTensor(w["k"], is_cuda=True)
    attn.v_proj, attn.o_proj = AGTensor(w["v"], is_cuda=True), AGTensor(w["o"], is_cuda=True)
    xt = AGTensor(x, is_cuda=True)
    for _ in range(3):
        attn(xt)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    reps = 20
    e0.record()
    for _ in range(reps):
        attn(xt)
    e1.record()
    torch.cuda.synchronize()
    ms = e0.elapsed_time(e1) / reps
    out = {"metric": "attention_layer_f32_ms", "value": ms, "unit": "ms", "higher_is_better": False, "dtype": "f32",
           "config": {"workload": "BASELINE config 1: one attention layer forward, fp32, S=128, hidden 2048, 32q/4kv "
                                  "heads, head_dim 64, device-resident tensors; 5 launches (4 projections + fused core)"}}
    try:
        from oracle import cref
        if os.path.exists(cref._GPU_SO):
            _, t = cref.gpu_gqa_layer(x, w["q"], w["k"], w["v"], w["o"], num_heads=32, num_kv_heads=4, head_dim=64,
                                      causal=True, time_iters=10, warmup=3)
            out["reference_cuda_ops_ms"] = float(t)
            out["reference_note"] = ("the reference's own operator sequence for the layer (5 op_mm, 2 op_rope, host-side "
                                     "head repeat, op_multiply, op_softmax) timed by its harness with CUDA events, "
                                     "oracle/_ref")
            out["speedup_vs_reference_cuda_ops"] = out["reference_cuda_ops_ms"] / ms
    except Exception as e:
        out["reference_cuda_ops_ms"] = None
        out["reference_note"] = repr(e)
    return out


def run_ours(args):
    import torch
    from baranet_bdml_b200 import ops, _lib
    _lib.load()   # fails loudly if the CUDA library is missing
    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    torch.cuda.set_device(local)
    dist = None
    if world > 1:
        import torch.distributed as dist_mod
        dist_mod.init_process_group("nccl", device_id=torch.device("cuda", local))
        dist = dist_mod
    pk = peaks()

    def reduce_max(x):
        if dist is None:
            return x
        t = torch.tensor([x], device="cuda", dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        return float(t.item())

    sampler = ClockSampler(local)
    if rank == 0:
        sampler.start()
    if args.decode_only:
        result = measure_decode(torch, args, rank, world, dist, reduce_max, pk)
    elif args.generate_only:
        result = measure_generate(torch, args, rank, world, dist, reduce_max, pk)
    elif args.longctx_only:
        result = measure_longctx(torch, args, rank, world, dist, reduce_max, pk)
    else:
        result = measure_prefill(torch, ops, args, rank, world, dist, reduce_max, pk)
        if not args.no_decode:
            try:
                result["decode"] = measure_decode(torch, args, rank, world, dist, reduce_max, pk)
            except Exception as e:  # the headline must still print
                result["decode"] = {"error": repr(e)}
            try:
                result["decode_long"] = measure_longctx(torch, args, rank, world, dist, reduce_max, pk)
            except Exception as e:
                result["decode_long"] = {"error": repr(e)}
            try:
                result["rmsnorm"] = measure_rmsnorm(torch, args, rank, world, dist, reduce_max, pk)
            except Exception as e:
                result["rmsnorm"] = {"error": repr(e)}
            try:
                result["embed_argmax"] = measure_embed_argmax(torch, args, rank, world, dist, reduce_max, pk)
            except Exception as e:
                result["embed_argmax"] = {"error": repr(e)}
            try:
                result["gemm"] = measure_gemm(torch, ops, args, rank, world, dist, reduce_max, pk)
            except Exception as e:
                result["gemm"] = {"error": repr(e)}
            try:
                result["mlp"] = measure_mlp(torch, ops, args, rank, world, dist, reduce_max, pk)
            except Exception as e:
                result["mlp"] = {"error": repr(e)}
            try:
                result["decoder_layer"] = measure_decoder_layer(torch, args, rank, world, dist, reduce_max, pk)
            except Exception as e:
                result["decoder_layer"] = {"error": repr(e)}
            if not args.no_generate:
                try:
                    result["generate"] = measure_generate(torch, args, rank, world, dist, reduce_max, pk)
                except Exception as e:
                    result["generate"] = {"error": repr(e)}
            if rank == 0 and world == 1:
                try:
                    result["layer_f32"] = measure_layer_f32(torch, args, rank, world, pk)
                except Exception as e:
                    result["layer_f32"] = {"error": repr(e)}
    if rank == 0:
        result["clocks"] = sampler.stop()
        if world == 1 and not args.no_cpu_baseline and not (args.decode_only or args.generate_only or args.longctx_only):
            r = cpu_prefill_sample(n_batches=2)
            result["cpu_baseline"] = {"value": r["value"], "unit": "TFLOP/s", "cores": r["cores"], "kind": "port",
                                      "sample": r["sample"], "seconds": r["seconds"]}
        # the partition of one config-2 batch over the ranks sits behind the headline keys
        if "sharded" in result:
            result["sharded"] = result.pop("sharded")
        # LAST key: the other half of the metric (decode) and the generation figures as flat scalars, so that a
        # reader of the end of the line sees them without walking the nested objects
        def pick(obj, *path):
            for k in path:
                if not isinstance(obj, dict) or k not in obj:
                    return None
                obj = obj[k]
            return obj
        if args.decode_only or args.generate_only or args.longctx_only:       # a run of one object: nothing to summarise
            _emit(json.dumps(result))
            if dist is not None:
                dist.destroy_process_group()
            return
        result["summary"] = {
            "prefill_tflops": result.get("value"), "prefill_frac": pick(result, "roofline", "frac"),
            "prefill_sharded_tflops": pick(result, "sharded", "value"),
            "decode_gbs": pick(result, "decode", "value"), "decode_ms": pick(result, "decode", "ms_per_step"),
            "decode_frac": pick(result, "decode", "roofline", "frac"),
            "decode_ms_eager": pick(result, "decode", "ms_per_step_eager"),
            "decode_sharded_gbs": pick(result, "decode", "sharded", "value"),
            "decode_sharded_ms": pick(result, "decode", "sharded", "ms_per_step"),
            "decode_long_gbs": pick(result, "decode_long", "value"), "decode_long_ms": pick(result, "decode_long", "ms_per_step"),
            "decode_long_ms_eager": pick(result, "decode_long", "ms_per_step_eager"),
            "decode_long_frac": pick(result, "decode_long", "roofline", "frac"),
            "decode_long_n": pick(result, "decode_long", "n_gpus"),
            "decode_long_max_abs_err": pick(result, "decode_long", "checks", "max_abs_err_partial_vs_fp32"),
            "generate_tokens_per_s": pick(result, "generate", "value"),
            "generate_prefill_ms": pick(result, "generate", "prefill_ms"),
            "generate_decode_ms_per_step": pick(result, "generate", "decode_ms_per_step"),
            "layer_f32_ms": pick(result, "layer_f32", "value"),
            "layer_f32_reference_cuda_ops_ms": pick(result, "layer_f32", "reference_cuda_ops_ms"),
        }
        _emit(json.dumps(result))
    if dist is not None:
        dist.destroy_process_group()


def run_design(name, args):
    """A model design's own measurements (bench_<name>.py) with the clocks seen meanwhile."""
    import importlib
    import torch
    torch.cuda.set_device(0)
    sampler = ClockSampler(0)
    sampler.start()
    res = importlib.import_module("bench_" + name).run(peaks(), max(10, args.steps))
    res["clocks"] = sampler.stop()
    _emit(json.dumps(res))


def main():
    # stdout carries exactly one JSON line: everything else that writes to file descriptor 1 (NCCL's version
    # banner, library chatter) is sent to stderr, and the line is written to the real stdout at the end
    real_stdout = os.fdopen(os.dup(1), "w")
    sys.stdout.flush()
    os.dup2(2, 1)
    global _emit
    def _emit(line):
        real_stdout.write(line + "\n")
        real_stdout.flush()
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=100)
    ap.add_argument("--warmup", type=int, default=10)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--no-cpu-baseline", action="store_true")
    ap.add_argument("--no-e2e", action="store_true", help="skip the host-buffer end-to-end measurement")
    ap.add_argument("--no-decode", action="store_true", help="skip the config-3 decode measurement")
    ap.add_argument("--no-generate", action="store_true", help="skip the config-5 generation measurement")
    ap.add_argument("--decode-only", action="store_true",
                    help="run only the decode measurement (for profiling); prints its object alone")
    ap.add_argument("--generate-only", action="store_true",
                    help="run only the config-5 generation (for profiling), one timed generation; prints its object alone")
    ap.add_argument("--generate-steps", type=int, default=128, help="decode steps of the config-5 generation")
    ap.add_argument("--longctx-only", action="store_true",
                    help="run only the config-4 sequence-split decode (decode kernel + exchange); prints its object alone")
    ap.add_argument("--soluzen", action="store_true",
                    help="measure the Soluzen design (whole models beside LLaMA, and its kernels one by one) instead of the "
                         "default workload; prints its object alone")
    ap.add_argument("--duponex", action="store_true", help="the same for the Duponex design")
    args = ap.parse_args()
    for design in ("soluzen", "duponex"):
        if getattr(args, design):
            run_design(design, args)
            return
    if args.warmup < 3 and args.impl == "ours":
        args.warmup = 3
    if args.impl == "reference":
        run_reference_arm(args)
    else:
        run_ours(args)


if __name__ == "__main__":
    main()
