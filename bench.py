#!/usr/bin/env python
"""Benchmark of the TernaSpMM hot path on B200.

Headline workload (the linear-layer sweep): the four ternary linears of a
BitNet-b1.58-2B decoder layer - QKV 2560->3840 (3 scale segments), O
2560->2560, gate-up 2560->13824 (2 segments), down 6912->2560 - for
``--layers`` layers with distinct random weights (30 layers = 410 MB of
compressed weights, more than three times the L2, so every call streams its
weights from HBM) at ``--tokens`` tokens.  One step = one pass over all
4 * layers linears.  Synthetic seeded inputs: weights i.i.d. over {-1,0,+1}
with P(0)=0.45, activations N(0,1) quantised per token to int8.

Prints ONE JSON line.  ``value`` = algorithmic bytes (compressed weights +
activations + scales + bf16 outputs) of all ranks per second with every input
resident in HBM, the step replayed as a CUDA graph; ``e2e`` = the same metric
through the Python call site (``TernaInfer_linear``) with the activations
copied from pinned host memory and the outputs copied back every step.
On one GPU the line also carries ``list_entry`` (the same step as ONE persistent
launch over a work list), ``by_tokens`` (the same sweep at 1 and 16 tokens),
``ref_kernels_b200`` (the reference's own small-batch CUDA kernels, built for
sm_100a from the reference checkout, timed in the same loop at 8, 16 and 64
tokens next to this library), ``lm_head`` (output head + greedy token),
``prefill`` (the large-batch paths against a bf16 GEMM and against the measured
int8 tensor-core issue rate) and ``decode`` (greedy decode tokens/s of the
30-layer model at batch 1 and 8).  On N > 1 GPUs the sweep runs as
independent replicas (the 2B model's 5 KV heads do not shard) and the line
carries ``tp``: the sharded linear stack of the 8192-wide model with one
collective per row-parallel linear, NCCL and fused.
``--impl reference`` times the CPU restatement of the reference's arithmetic
(the reference has no CPU implementation of this path and its CUDA library
does not build without an un-vendored CUTLASS) on the host cores.
"""
import argparse
import ctypes
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

import numpy as np

SHAPES = [  # name, N, K, ws_num
    ("wqkv", 3840, 2560, 3),
    ("wo", 2560, 2560, 1),
    ("w13", 13824, 2560, 2),
    ("w2", 2560, 6912, 1),
]
P_ZERO = 0.45


def measured_peak():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        try:
            return float(json.load(open(path))["hbm_gbs"]), "measured"
        except Exception:
            pass
    return 6650.0, "fallback"


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed
    region runs."""
    FIELDS = ("index,clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,"
              "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
              "clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_index):
        self.gpu = gpu_index
        self.proc = None
        self.lines = []

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", str(self.gpu), "--query-gpu=" + self.FIELDS, "--format=csv,noheader,nounits",
                 "-lms", "100"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except Exception:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.lines.append(line.strip())

    def stop(self):
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except Exception:
            self.proc.kill()
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for ln in self.lines:
            f = [x.strip() for x in ln.split(",")]
            if len(f) < 7:
                continue
            try:
                sm.append(float(f[1]))
                mx.append(float(f[2]))
            except ValueError:
                continue
            for n, v in zip(names, f[3:7]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        return {"sm_mhz": float(np.median(sm)) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "samples": len(sm), "reasons": sorted(reasons)}


# ----------------------------------------------------------------------------
# CPU arm: the oracle port timed on the host cores (checker code, used here
# only as the thing to compare against, never on the GPU arm's path).
# ----------------------------------------------------------------------------

def ncu_traffic(kernel, tokens):
    """dram__bytes_read.sum + dram__bytes_write.sum per launch of ``kernel`` at ``tokens`` tokens,
    averaged over the step's launches, from the table that is written next to the ncu summaries
    when a capture is processed (profiles/ncu_traffic.json); None when there is no entry."""
    path = os.path.join(ROOT, "profiles", "ncu_traffic.json")
    try:
        return float(json.load(open(path))[kernel][str(tokens)])
    except Exception:
        return None


def sweep_config(args, world):
    """The workload description both arms print (the driver compares them)."""
    return {"workload": f"bitnet2b_linear_sweep_M{args.tokens}", "tokens": args.tokens, "layers": args.layers,
            "linears_per_step": 4 * args.layers, "p_zero": P_ZERO, "seed": args.seed,
            "l2_policy": "inputs larger than L2: each step streams the distinct compressed weights of all layers "
                         "(410 MB at 30 layers)",
            "parallelism": "replicas only" if world > 1 else "single GPU"}


def cpu_sample(tokens, seconds_budget, seed=1234):
    sys.path.insert(0, os.path.join(ROOT, "oracle"))
    import ternaspmm_oracle as o
    import c_oracle
    lib = c_oracle.load()
    lib.oracle_set_num_threads(os.cpu_count() or 1)    # launchers export OMP_NUM_THREADS=1; use the host's cores
    cores = int(lib.oracle_num_threads())
    items, alg = [], 0
    for li, (name, N, K, ws_num) in enumerate(SHAPES):
        rng = np.random.default_rng(seed + li)
        w = (rng.random((N, K), dtype=np.float32) >= P_ZERO).astype(np.int8)
        w *= (rng.integers(0, 2, size=(N, K), dtype=np.int8) * 2 - 1)
        xq, s = o.make_activations(tokens, K, seed + 100 + li)
        ws = o.make_ws(ws_num, seed + 200 + li)
        nnz = int(np.count_nonzero(w))
        tiles = N * K // 4096
        wbytes = N * K // 8 + (nnz + 16 * tiles) // 8 + 4 * (tiles + 1) + 6 * tiles   # padding estimated at 16 bits/tile
        alg += wbytes + tokens * K + 2 * tokens + 8 + 2 * tokens * N
        items.append((xq, w, o.f32_to_bf16_bits(s.reshape(-1)), o.f32_to_bf16_bits(ws), ws_num))
    def one_pass():
        for xq, w, sb, wb, ws_num in items:
            c_oracle.ternaspmm(xq, w, sb, wb, ws_num)
    one_pass()
    t0 = time.perf_counter()
    one_pass()
    dt = time.perf_counter() - t0
    reps = max(1, min(2000, int(seconds_budget / max(dt, 1e-6))))
    return one_pass, alg, cores, reps, dt


def run_reference_arm(args):
    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    if rank != 0:
        return
    # a step = a bounded sample of the sweep (some passes over one layer); the whole run stays near a minute.
    # The value is what ALL host cores of the box deliver, whatever N is: there is one host.
    one_pass, alg, cores, reps, _ = cpu_sample(args.tokens, max(0.1, 60.0 / max(1, args.steps)))
    for _ in range(args.warmup):
        one_pass()
    t0 = time.perf_counter()
    for _ in range(args.steps):
        for _ in range(reps):
            one_pass()
    dt = time.perf_counter() - t0
    val = alg * reps * args.steps / dt / 1e9
    sample = (f"{reps} passes over one layer (4 linears) per step at {args.tokens} tokens, dense ternary int8 weights; "
              "CPU restatement of the reference arithmetic (C, OpenMP) - the reference has no CPU path")
    line = {
        "impl": "reference", "metric": "ternaspmm_algorithmic_GBps", "value": val, "unit": "GB/s",
        "n_gpus": world, "steps": args.steps, "warmup": args.warmup, "ms_per_step": dt / args.steps * 1e3,
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "int8xternary->int32->bf16",
        "data": "synthetic", "config": sweep_config(args, world),
        "cpu_baseline": {"value": val, "unit": "GB/s", "cores": cores, "kind": "port", "sample": sample},
        "e2e": {"value": val, "unit": "GB/s", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
        "gpu_launches": 0,
    }
    print(json.dumps(line))


# ----------------------------------------------------------------------------
# GPU arm
# ----------------------------------------------------------------------------

def build_workload(torch, layers, seed, device):
    """The packed weights of `layers` layers (distinct seeded random ternary matrices)."""
    from ternainfer_b200.convert import compress_weight, compressed_nbytes
    gen = torch.Generator(device=device)
    work, wbytes_total = [], 0
    for layer in range(layers):
        for si, (name, N, K, ws_num) in enumerate(SHAPES):
            gen.manual_seed(seed + 1000 * layer + si)
            r = torch.rand((N, K), generator=gen, device=device)
            sign = (torch.randint(0, 2, (N, K), generator=gen, device=device, dtype=torch.int8) * 2 - 1)
            w = torch.where(r < P_ZERO, torch.zeros((), dtype=torch.int8, device=device), sign)
            cv, tg, tm, bm = compress_weight(w)
            nbytes = compressed_nbytes(cv, tg, tm, bm)
            ws = torch.zeros(4, device=device)
            ws[:ws_num] = torch.rand(ws_num, generator=gen, device=device) * 0.04 + 0.01
            item = dict(name=name, N=N, K=K, ws_num=ws_num, cv=cv, tg=tg, tm=tm, bm=bm, ws=ws.to(torch.bfloat16),
                        wbytes=nbytes)
            if layer == 0:
                item["dense"] = w.cpu().numpy()
            work.append(item)
            wbytes_total += nbytes
            del w, r, sign
    return work, wbytes_total


def algorithmic_bytes(it, tokens):
    """Compressed weight + int8 activations + per-token scales + weight scales + bf16 outputs of one call."""
    return it["wbytes"] + tokens * it["K"] + 2 * tokens + 8 + 2 * tokens * it["N"]


class Env:
    """Process-wide state of a GPU run."""

    def __init__(self):
        import torch
        import torch.distributed as dist
        self.torch, self.dist = torch, dist
        self.world = int(os.environ.get("WORLD_SIZE", "1"))
        self.rank = int(os.environ.get("RANK", "0"))
        self.local_rank = int(os.environ.get("LOCAL_RANK", "0"))
        if not torch.cuda.is_available():
            raise SystemExit("bench.py needs a CUDA GPU: the TernaSpMM library has no CPU path")
        torch.cuda.set_device(self.local_rank)
        self.device = torch.device("cuda", self.local_rank)
        if self.world > 1:
            os.environ.setdefault("TORCH_SYMM_MEM_DISABLE_MULTICAST", "1")   # peer memory by plain loads/stores only
            dist.init_process_group("nccl", device_id=self.device)
        from ternainfer_b200 import load_library
        self.lib = load_library()   # raises if the CUDA library is missing
        self.stream = torch.cuda.Stream(device=self.device)

    def barrier(self):
        self.torch.cuda.synchronize()
        if self.world > 1:
            self.dist.barrier()
            self.torch.cuda.synchronize()

    def max_over_ranks(self, ms):
        t = self.torch.tensor([ms], dtype=self.torch.float64, device=self.device)
        if self.world > 1:
            self.dist.all_reduce(t, op=self.dist.ReduceOp.MAX)
        return float(t.item())

    def time_replays(self, replay, steps, warmup, min_load_s=0.0):
        """`warmup` untimed replays (plus, with min_load_s, enough further ones to keep the GPU under
        this load for that long, so that the clock sampler sees it), then EXACTLY `steps` timed ones
        between CUDA events on the launching stream, barrier + synchronize on both sides; max over ranks."""
        torch = self.torch
        with torch.cuda.stream(self.stream):
            for _ in range(warmup):
                replay()
            if min_load_s > 0:
                self.stream.synchronize()
                t0 = time.perf_counter()
                replay()
                self.stream.synchronize()
                one = max(time.perf_counter() - t0, 1e-6)
                extra = min(20000, int(min_load_s / one))
                if self.world > 1:   # the same count on every rank: the replayed graph may hold collectives
                    cnt = torch.tensor([extra], dtype=torch.int64, device=self.device)
                    self.dist.broadcast(cnt, 0)
                    extra = int(cnt.item())
                for _ in range(extra):
                    replay()
            self.barrier()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record(self.stream)
            for _ in range(steps):
                replay()
            e1.record(self.stream)
            self.barrier()
        return self.max_over_ranks(e0.elapsed_time(e1))


def quantised_inputs(env, M, seed):
    torch = env.torch
    from ternainfer_b200.linear import quant_input
    gen = torch.Generator(device="cpu").manual_seed(seed + 5)
    x_host = {K: torch.randn((M, K), generator=gen).to(torch.bfloat16).pin_memory() for K in (2560, 6912)}
    xq, s = {}, {}
    for K, xh in x_host.items():
        xq[K], s[K] = quant_input(xh.to(env.device))
        s[K] = s[K].contiguous()
    return xq, s


def check_layer0_against_oracle(env, work, outs, xq, s):
    """Sanity check outside the timed region: the first layer's outputs against the CPU oracle."""
    torch = env.torch
    sys.path.insert(0, os.path.join(ROOT, "oracle"))
    import ternaspmm_oracle as o
    for it, out in zip(work[:len(SHAPES)], outs[:len(SHAPES)]):
        K = it["K"]
        want = o.ternaspmm(xq[K].cpu().numpy(), it["dense"], s[K].float().cpu().numpy().reshape(-1),
                           it["ws"].float().cpu().numpy(), it["ws_num"])
        got = out.view(torch.int16).cpu().numpy().view(np.uint16)
        if not (got == want).all():
            raise SystemExit(f"bench sanity check failed for {it['name']}: GPU result differs from the oracle")
    if env.lib.ternaspmm_last_status() != 0:
        raise SystemExit("bench: library reported a non-zero status")


def sweep_leg(env, work, M, args, headline):
    """One pass over all linears at M tokens per step, inputs resident in HBM, the step replayed as one
    CUDA graph.  Returns value / ms_per_step / roofline for that token count."""
    torch, lib = env.torch, env.lib
    xq, s = quantised_inputs(env, M, args.seed)
    outs = [torch.empty((M, it["N"]), dtype=torch.bfloat16, device=env.device) for it in work]
    alg_step = sum(algorithmic_bytes(it, M) for it in work)

    def launch_all():
        st = torch.cuda.current_stream().cuda_stream
        for it, out in zip(work, outs):
            K = it["K"]
            lib.bitlinear_TernaSpMM(xq[K].data_ptr(), it["bm"].data_ptr(), it["tg"].data_ptr(), it["tm"].data_ptr(),
                                    it["cv"].data_ptr(), out.data_ptr(), s[K].data_ptr(), it["ws"].data_ptr(),
                                    it["ws_num"], M, it["N"], K, 7, 0, st)

    with torch.cuda.stream(env.stream):
        launch_all()
    env.stream.synchronize()
    check_layer0_against_oracle(env, work, outs, xq, s)
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.stream(env.stream):
        with torch.cuda.graph(graph, stream=env.stream):
            launch_all()
    ms = env.time_replays(graph.replay, args.steps, args.warmup, min_load_s=1.0 if headline else 0.2)
    peak, peak_kind = measured_peak()
    launches = len(work)
    per_launch_us = ms * 1e3 / (args.steps * launches)
    achieved = (alg_step / launches) / (per_launch_us * 1e-6) / 1e9
    res = {"value": alg_step * env.world * args.steps / (ms * 1e-3) / 1e9, "unit": "GB/s",
           "ms_per_step": ms / args.steps,
           "roofline": {"bound": "hbm", "achieved": achieved, "peak": peak, "unit": "GB/s", "frac": achieved / peak,
                        "peak_kind": "of " + peak_kind, "frac_of_nominal_8000": achieved / 8000.0,
                        "kernel": "spmm_small_m_kernel", "avg_launch_us": per_launch_us,
                        "algorithmic_bytes_per_launch": alg_step / launches,
                        "traffic": ncu_traffic("spmm_small_m_kernel", M)},
           "gpu_launches": launches * args.steps}
    return res, (xq, s, alg_step)


def e2e_leg(env, work, M, args, xq, s, alg_step):
    """The same step through the Python call site with HOST buffers: this step's activations come from
    pinned host memory, every output goes back to pinned host memory (on a side stream that forks after
    its producer, so the copies overlap the following linears).  Captured once, exactly as the reference's
    generate.py captures its forward; a step is one replay."""
    torch = env.torch
    from ternainfer_b200.linear import TernaInfer_linear
    xq_host = {K: v.cpu().pin_memory() for K, v in xq.items()}
    s_host = {K: v.cpu().pin_memory() for K, v in s.items()}
    out_host = [torch.empty((M, it["N"]), dtype=torch.bfloat16).pin_memory() for it in work]
    xq_dev = {K: torch.empty_like(v, device=env.device) for K, v in xq_host.items()}
    s_dev = {K: torch.empty_like(v, device=env.device) for K, v in s_host.items()}
    h2d = sum(v.numel() * v.element_size() for v in xq_host.values()) + \
        sum(v.numel() * v.element_size() for v in s_host.values())
    d2h = sum(v.numel() * v.element_size() for v in out_host)
    keep = []
    graph = torch.cuda.CUDAGraph()
    side = torch.cuda.Stream(device=env.device)
    with torch.cuda.stream(env.stream):
        with torch.cuda.graph(graph, stream=env.stream):
            for K in xq_host:
                xq_dev[K].copy_(xq_host[K], non_blocking=True)
                s_dev[K].copy_(s_host[K], non_blocking=True)
            for it, oh in zip(work, out_host):
                K = it["K"]
                y = TernaInfer_linear(xq_dev[K], it["cv"], it["tg"], it["tm"], it["bm"], None, s_dev[K],
                                      it["ws"], it["ws_num"], it["N"])
                keep.append(y)
                done = torch.cuda.Event()
                done.record(env.stream)
                side.wait_event(done)
                with torch.cuda.stream(side):
                    oh.copy_(y, non_blocking=True)
            joined = torch.cuda.Event()
            joined.record(side)
            env.stream.wait_event(joined)
    ms = env.time_replays(graph.replay, args.steps, max(3, args.warmup))
    return {"value": alg_step * env.world * args.steps / (ms * 1e-3) / 1e9, "unit": "GB/s",
            "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": d2h, "ms_per_step": ms / args.steps,
            "api": "ternainfer_b200.linear.TernaInfer_linear captured in a CUDA graph together with its H2D and "
                   "(side-stream) D2H copies; one replay per step"}


def ref_kernels_leg(env, work, args):
    """The reference's own small-batch CUDA kernels (SpMM + split-K reduction, SPLIT_K = 7 as model.py
    passes it), compiled for sm_100a from the reference checkout into oracle/_ref, next to this library
    in the same loop: one pass over `layers` x 4 linears per step, every call on its own copy of the
    packed weights so that all of them stream from HBM.  The reference supports 8, 16, 32 and 64 tokens."""
    torch = env.torch
    so = os.path.join(ROOT, "oracle", "_ref", "libternaspmm_ref_decode.so")
    if not os.path.exists(so):
        return {"unavailable": "oracle/_ref/libternaspmm_ref_decode.so not built (needs the reference checkout)"}
    sys.path.insert(0, os.path.join(ROOT, "oracle"))
    import ternaspmm_oracle as o
    ref = ctypes.CDLL(so)
    P, I = ctypes.c_void_p, ctypes.c_int
    ref.ref_bitlinear_TernaSpMM_decode.argtypes = [P] * 8 + [I] * 5 + [P, P]
    ref.ref_bitlinear_TernaSpMM_decode.restype = I

    def dev(a):
        return torch.from_numpy(np.ascontiguousarray(a).view(np.uint8).reshape(-1).copy()).to(env.device)

    layers = len(work) // len(SHAPES)
    packed = []   # per shape: `layers` device copies of the reference-layout arrays of layer 0's weight
    for it in work[:len(SHAPES)]:
        cv, tg, tm, bm = o.compress_weight_ref(it["dense"])
        cv = np.concatenate([cv, np.zeros(16, np.uint32)])        # the reference kernels prefetch past the ends
        tg = np.concatenate([tg, np.full(8, tg[-1], np.int32)])
        tm = np.concatenate([tm, np.zeros(16, np.uint16)])
        base = [dev(a) for a in (bm, tg, tm, cv)]
        packed.append([base] + [[t.clone() for t in base] for _ in range(layers - 1)])
    out = {"split_k": 7, "layers": layers, "note": "same weights, activations and scales on both sides; ours = "
           "bitlinear_TernaSpMM of this library; reference = mySpMM_Kernel_bitmap_v3 + SplitK_Reduction"}
    for M in (8, 16, 64):
        xq, s = quantised_inputs(env, M, args.seed)
        outs = [torch.empty((M, it["N"]), dtype=torch.bfloat16, device=env.device) for it in work[:len(SHAPES)]]
        wsp = torch.zeros(7 * M * 13824, dtype=torch.int32, device=env.device)

        def launch_ref():
            st = torch.cuda.current_stream().cuda_stream
            for layer in range(layers):
                for si, it in enumerate(work[:len(SHAPES)]):
                    bm, tg, tm, cv = packed[si][layer]
                    K = it["K"]
                    rc = ref.ref_bitlinear_TernaSpMM_decode(xq[K].data_ptr(), bm.data_ptr(), tg.data_ptr(), tm.data_ptr(),
                                                            cv.data_ptr(), outs[si].data_ptr(), s[K].data_ptr(),
                                                            it["ws"].data_ptr(), it["ws_num"], M, it["N"], K, 7,
                                                            wsp.data_ptr(), st)
                    if rc != 0:
                        raise SystemExit(f"reference kernels: CUDA error {rc}")

        ours_outs = [torch.empty((M, it["N"]), dtype=torch.bfloat16, device=env.device) for it in work]

        def launch_ours():
            st = torch.cuda.current_stream().cuda_stream
            for it, o_ in zip(work, ours_outs):
                K = it["K"]
                env.lib.bitlinear_TernaSpMM(xq[K].data_ptr(), it["bm"].data_ptr(), it["tg"].data_ptr(),
                                            it["tm"].data_ptr(), it["cv"].data_ptr(), o_.data_ptr(), s[K].data_ptr(),
                                            it["ws"].data_ptr(), it["ws_num"], M, it["N"], K, 7, 0, st)

        res = {}
        for name, fn in (("reference", launch_ref), ("ours", launch_ours)):
            with torch.cuda.stream(env.stream):
                fn()
            env.stream.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.stream(env.stream):
                with torch.cuda.graph(g, stream=env.stream):
                    fn()
            ms = env.time_replays(g.replay, args.steps, args.warmup)
            res[name + "_ms_per_step"] = ms / args.steps
        # layer 0: both sides must agree bit for bit
        same = all(torch.equal(a, b) for a, b in zip(outs, ours_outs[:len(SHAPES)]))
        alg = sum(algorithmic_bytes(it, M) for it in work)
        res.update({"reference_GBps": alg / (res["reference_ms_per_step"] * 1e-3) / 1e9,
                    "ours_GBps": alg / (res["ours_ms_per_step"] * 1e-3) / 1e9,
                    "speedup": res["reference_ms_per_step"] / res["ours_ms_per_step"], "outputs_identical": bool(same)})
        out[str(M)] = res
        del wsp
    return out


def list_leg(env, work, M, args):
    """The same step through the work-list entry points: all linears of the step in ONE persistent
    launch (ternaspmm_list_run), inputs resident in HBM, replayed as a CUDA graph."""
    torch, lib = env.torch, env.lib
    from ternainfer_b200.lib import ListItem
    xq, s = quantised_inputs(env, M, args.seed)
    outs = [torch.empty((M, it["N"]), dtype=torch.bfloat16, device=env.device) for it in work]
    arr = (ListItem * len(work))()
    for a, it, out in zip(arr, work, outs):
        K = it["K"]
        a.x, a.bitmap, a.tile_offsets, a.quarter_offsets = xq[K].data_ptr(), it["bm"].data_ptr(), it["tg"].data_ptr(), it["tm"].data_ptr()
        a.sign_words, a.out, a.s, a.ws, a.residual = it["cv"].data_ptr(), out.data_ptr(), s[K].data_ptr(), it["ws"].data_ptr(), None
        a.ws_num, a.M, a.N, a.K, a.seg1, a.seg2, a.seg3, a.prefill_form = it["ws_num"], M, it["N"], K, 0, 0, 0, -1
    tb, sb = ctypes.c_longlong(), ctypes.c_longlong()
    entries = lib.ternaspmm_list_plan(arr, len(work), ctypes.byref(tb), ctypes.byref(sb))
    if entries < 0:
        raise SystemExit("bench: the work list was rejected")
    table = torch.empty(tb.value, dtype=torch.uint8, device=env.device)
    scratch = torch.empty(sb.value, dtype=torch.uint8, device=env.device)
    with torch.cuda.stream(env.stream):
        handle = lib.ternaspmm_list_create(arr, len(work), table.data_ptr(), scratch.data_ptr(), env.stream.cuda_stream)
        if not handle:
            raise SystemExit("bench: could not create the work list")
        lib.ternaspmm_list_run(handle, env.stream.cuda_stream)
    env.stream.synchronize()
    check_layer0_against_oracle(env, work, outs, xq, s)
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.stream(env.stream):
        with torch.cuda.graph(graph, stream=env.stream):
            lib.ternaspmm_list_run(handle, env.stream.cuda_stream)
    ms = env.time_replays(graph.replay, args.steps, args.warmup, min_load_s=0.3)
    if lib.ternaspmm_last_status() != 0:
        raise SystemExit("bench: the work-list run reported a non-zero status")
    lib.ternaspmm_list_destroy(handle)
    alg_step = sum(algorithmic_bytes(it, M) for it in work)
    peak, peak_kind = measured_peak()
    achieved = alg_step * args.steps / (ms * 1e-3) / 1e9
    return {"value": achieved * env.world, "unit": "GB/s", "ms_per_step": ms / args.steps, "items": len(work),
            "entries": entries, "tokens": M,
            "api": "ternaspmm_list_run: one persistent launch per step over all of the step's linears",
            "roofline": {"bound": "hbm", "achieved": achieved, "peak": peak, "unit": "GB/s", "frac": achieved / peak,
                         "peak_kind": "of " + peak_kind, "frac_of_nominal_8000": achieved / 8000.0,
                         "kernel": "spmm_list_kernel", "avg_launch_us": ms * 1e3 / args.steps,
                         "avg_item_us": ms * 1e3 / args.steps / len(work), "algorithmic_bytes_per_launch": alg_step,
                         "traffic": ncu_traffic("spmm_list_kernel", M)},
            "gpu_launches": args.steps}


def lm_head_leg(env, args):
    """The output-head kernel alone: logits-free greedy token of M rows over the 128256 x 2560 bf16
    embedding (657 MB, five times the L2: every call streams it from HBM)."""
    torch, lib = env.torch, env.lib
    V, K = 128256, 2560
    g = torch.Generator(device=env.device).manual_seed(args.seed)
    emb = (0.02 * torch.randn((V, K), generator=g, device=env.device)).to(torch.bfloat16)
    scratch = torch.zeros(int(lib.ternaspmm_lm_head_scratch_bytes()), dtype=torch.uint8, device=env.device)
    peak, peak_kind = measured_peak()
    out = {}
    for M in (1, 8):
        h = torch.randn((M, K), generator=g, device=env.device).to(torch.bfloat16)
        toks = torch.empty(M, dtype=torch.int64, device=env.device)

        def run():
            lib.ternaspmm_lm_head_argmax(h.data_ptr(), emb.data_ptr(), M, V, K, None, toks.data_ptr(), 1,
                                         scratch.data_ptr(), torch.cuda.current_stream().cuda_stream)

        with torch.cuda.stream(env.stream):
            run()
        env.stream.synchronize()
        want = torch.nn.functional.linear(h, emb).float()
        picked = want.gather(1, toks.view(-1, 1)).view(-1)
        if not (want.max(dim=1).values - picked <= want.abs().max() * 2.0 ** -6).all():
            raise SystemExit("bench: the head kernel's greedy tokens disagree with the dense product")
        ms = env.time_replays(run, args.steps, args.warmup)
        nbytes = V * K * 2 + M * K * 2 + 8 * M
        gbs = nbytes * args.steps / (ms * 1e-3) / 1e9
        dense_ms = env.time_replays(lambda: torch.nn.functional.linear(h, emb).float().argmax(-1), args.steps, args.warmup)
        out[str(M)] = {"us_per_call": ms * 1e3 / args.steps, "GBps": gbs, "frac": gbs / peak, "peak_kind": "of " + peak_kind,
                       "algorithmic_bytes": nbytes, "torch_bf16_linear_plus_argmax_us": dense_ms * 1e3 / args.steps}
    del emb
    torch.cuda.empty_cache()
    return out


def prefill_leg(env, args, token_counts=(256, 1024, 2048, 4096)):
    """Large-batch calls on the gate-up layer (13824 x 2560, the largest of the sweep): the tcgen05 kernel that
    decodes on chip, the path through the reference-sized workspace (decompress once, then tcgen05 on CTA pairs
    with both operands by TMA; `auto` names the one the library picks by itself) and torch's dense bf16 linear on the de-quantised weight (cuBLAS: the comparator of the reference's own kernel
    test).  One weight, launched back to back: the 7 MB of compressed weight stay in L2, as in that test."""
    torch, lib = env.torch, env.lib
    from ternainfer_b200.convert import compress_weight
    N, K, ws_num = 13824, 2560, 2
    g = torch.Generator(device=env.device).manual_seed(args.seed)
    r = torch.rand((N, K), generator=g, device=env.device)
    sign = torch.randint(0, 2, (N, K), generator=g, device=env.device, dtype=torch.int8) * 2 - 1
    w = torch.where(r < P_ZERO, torch.zeros((), dtype=torch.int8, device=env.device), sign)
    cv, tg, tm, bm = compress_weight(w)
    wd = w.to(torch.bfloat16)
    ws = torch.tensor([0.02, 0.03, 0.0, 0.0]).to(torch.bfloat16).to(env.device)
    work = torch.empty(N * K, dtype=torch.int8, device=env.device)
    peak_tf = None
    try:
        peak_tf = float(json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json")))["bf16_tflops"])
    except Exception:
        pass
    rate = float(lib.ternaspmm_debug_int8_mma_rate(6400, torch.cuda.current_stream().cuda_stream)) / 1e12
    out = {"layer": "gate-up 13824x2560", "note": "int8 tensor-core ops 2*M*N*K per call; frac_of_measured_bf16_peak is of "
           "the measured bf16 cuBLAS burst peak, frac_of_int8_issue_rate of the rate at which this GPU issues tcgen05 int8 "
           "MMAs from resident operands (measured here, one CTA per SM)",
           "int8_mma_issue_rate_TOPs": rate}
    for M in token_counts:
        xq = torch.randint(-127, 128, (M, K), dtype=torch.int8, device=env.device)
        sc = (torch.rand(M, device=env.device) * 50 + 1).to(torch.bfloat16)
        y = torch.empty((M, N), dtype=torch.bfloat16, device=env.device)
        xb = xq.to(torch.bfloat16)

        def call(path):
            lib.bitlinear_TernaSpMM_ws(xq.data_ptr(), bm.data_ptr(), tg.data_ptr(), tm.data_ptr(), cv.data_ptr(), y.data_ptr(),
                                       sc.data_ptr(), ws.data_ptr(), ws_num, M, N, K, None, work.data_ptr(), N * K, path,
                                       torch.cuda.current_stream().cuda_stream)

        t_chip = env.time_replays(lambda: call(1), args.steps, args.warmup) / args.steps * 1e3
        a = y.clone()
        t_ws = env.time_replays(lambda: call(2), args.steps, args.warmup) / args.steps * 1e3
        if not torch.equal(a, y):
            raise SystemExit("bench: the two large-batch paths disagree")
        t_torch = env.time_replays(lambda: torch.nn.functional.linear(xb, wd), args.steps, args.warmup) / args.steps * 1e3
        call(0)
        shape = (ctypes.c_int * 6)()
        lib.ternaspmm_last_launch_shape(shape)
        ops = 2.0 * M * N * K
        best = min(t_chip, t_ws)
        out[str(M)] = {"on_chip_us": t_chip, "workspace_us": t_ws, "auto": "workspace" if shape[0] in (6, 7) else "on_chip",
                       "torch_bf16_linear_us": t_torch,
                       "tensor_TOPs": ops / best / 1e6, "frac_of_measured_bf16_peak": (ops / best / 1e6 / peak_tf) if peak_tf else None,
                       "frac_of_int8_issue_rate": (ops / best / 1e6 / rate) if rate > 0 else None,
                       "speedup_vs_torch_bf16": t_torch / best}
    del w, wd, work
    torch.cuda.empty_cache()
    return out


def run_single_leg(args):
    """--workload list | head | prefill: one leg on its own (short runs for profiling)."""
    env = Env()
    if args.workload == "list":
        work, _ = build_workload(env.torch, args.layers, args.seed + 7919 * env.rank, env.device)
        res = list_leg(env, work, args.tokens, args)
        line = {"metric": "ternaspmm_algorithmic_GBps", "value": res["value"], "unit": "GB/s", "n_gpus": env.world,
                "steps": args.steps, "warmup": args.warmup, "ms_per_step": res["ms_per_step"], "higher_is_better": True,
                "scaling": "weak", "vs_baseline": None, "dtype": "int8xternary->int32->bf16", "data": "synthetic",
                "config": dict(sweep_config(args, env.world), entry="ternaspmm_list_run"), "roofline": res["roofline"],
                "gpu_launches": res["gpu_launches"]}
    elif args.workload == "head":
        res = lm_head_leg(env, args)
        line = {"metric": "lm_head_GBps", "value": res["8"]["GBps"], "unit": "GB/s", "n_gpus": 1, "steps": args.steps,
                "warmup": args.warmup, "ms_per_step": res["8"]["us_per_call"] / 1e3, "higher_is_better": True,
                "config": {"workload": "lm_head_argmax_128256x2560_M8"}, "lm_head": res, "gpu_launches": args.steps}
    else:
        res = prefill_leg(env, args, (args.tokens,) if args.tokens > 64 else (2048,))
        key = [k for k in res if k.isdigit()][0]
        line = {"metric": "prefill_int8_TOPs", "value": res[key]["tensor_TOPs"], "unit": "TOP/s", "n_gpus": 1,
                "steps": args.steps, "warmup": args.warmup, "higher_is_better": True,
                "config": {"workload": f"gate_up_13824x2560_M{key}"}, "prefill": res, "gpu_launches": 2 * args.steps}
    if env.rank == 0:
        print(json.dumps(line), flush=True)
    _finish(env.world)


def run_gpu_arm(args):
    env = Env()
    torch = env.torch
    M = args.tokens
    work, wbytes_total = build_workload(torch, args.layers, args.seed + 7919 * env.rank, env.device)
    sampler = ClockSampler(env.local_rank)
    if env.rank == 0:
        sampler.start()
    head, (xq, s, alg_step) = sweep_leg(env, work, M, args, headline=True)
    e2e = e2e_leg(env, work, M, args, xq, s, alg_step)
    clocks = sampler.stop() if env.rank == 0 else None

    def guarded(fn, *a):
        """The further legs of a one-GPU run must not cost the headline line: a leg that cannot run here
        (a library of the attention glue missing, memory) is reported as an error object.  A leg that finds
        WRONG results ends the run (SystemExit is not caught)."""
        try:
            return fn(*a)
        except Exception as e:      # noqa: BLE001
            torch.cuda.synchronize()
            return {"error": f"{type(e).__name__}: {e}"[:300]}

    extras = {}
    if not args.headline_only:
        if M <= 16:
            extras["list_entry"] = list_leg(env, work, M, args) if env.world > 1 else guarded(list_leg, env, work, M, args)
        if env.world == 1:
            extras["by_tokens"] = {}
            for m in (1, 16):
                if m != M:
                    def both(m=m):
                        r = sweep_leg(env, work, m, args, headline=False)[0]
                        r["list_entry"] = list_leg(env, work, m, args)
                        return r
                    extras["by_tokens"][str(m)] = guarded(both)
            extras["ref_kernels_b200"] = guarded(ref_kernels_leg, env, work, args)
        del work
        torch.cuda.empty_cache()
        if env.world == 1:
            extras["lm_head"] = guarded(lm_head_leg, env, args)
            extras["prefill"] = guarded(prefill_leg, env, args)
            extras["decode"] = guarded(decode_leg, args)
        else:
            extras["tp"] = {mode: tp_stack(env, args, mode, 64, 4) for mode in ("single", "fused")}

    if env.rank == 0:
        cpu_baseline = None            # timed at N = 1 only (rank 0's host cores)
        if env.world == 1:
            one_pass, cpu_alg, cores, reps, dt = cpu_sample(M, 10.0)
            t0 = time.perf_counter()
            for _ in range(reps):
                one_pass()
            cpu_dt = time.perf_counter() - t0
            cpu_baseline = {"value": cpu_alg * reps / cpu_dt / 1e9, "unit": "GB/s", "cores": cores, "kind": "port",
                            "sample": f"{reps} passes over one layer (4 linears) at {M} tokens, dense int8 ternary "
                                      f"weights, {cpu_dt:.1f} s"}
        line = {
            "metric": "ternaspmm_algorithmic_GBps", "value": head["value"], "unit": "GB/s", "n_gpus": env.world,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": head["ms_per_step"],
            "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
            "dtype": "int8xternary->int32->bf16", "data": "synthetic",
            "config": sweep_config(args, env.world),
            "launch": "one CUDA graph replay per step", "compressed_weight_bytes_per_rank": wbytes_total,
            "roofline": head["roofline"], "cpu_baseline": cpu_baseline, "e2e": e2e,
            "gpu_launches": head["gpu_launches"], "clocks": clocks,
        }
        line.update(extras)
        print(json.dumps(line), flush=True)
    _finish(env.world)


# ----------------------------------------------------------------------------
# Tensor-parallel arm (the scaled ternary model): hidden 8192, 64/8 heads,
# ffn 28672, batch 64.  Per layer: QKV and gate-up column-parallel, O and down
# row-parallel with ONE all-reduce each; the attention itself is not part of
# the path and is skipped (its output is a fixed synthetic tensor).  Strong
# scaling: the model is fixed, each rank holds 1/N of every weight.
# ----------------------------------------------------------------------------

def tp_stack(env, args, mode, M, L):
    """`L` layers of the 8192-wide model's four linears at `M` tokens, sharded over all ranks (see the
    comment above).  Returns the timing of one step (all layers) as a dict."""
    torch, dist = env.torch, env.dist
    from ternainfer_b200 import tp
    from ternainfer_b200.convert import compress_weight, compressed_nbytes
    world, rank, device = env.world, env.rank, env.device
    dim, H, Hkv, D, ffn = 8192, 64, 8, 128, 28672
    gen = torch.Generator(device=device)

    def tern(n, k, seed):
        gen.manual_seed(seed)
        r = torch.rand((n, k), generator=gen, device=device)
        sign = torch.randint(0, 2, (n, k), generator=gen, device=device, dtype=torch.int8) * 2 - 1
        return torch.where(r < P_ZERO, torch.zeros((), dtype=torch.int8, device=device), sign)

    layers, wbytes, dense0 = [], 0, {}
    for li in range(L):
        dic = {}
        specs = [("wqkv", "column", (H + 2 * Hkv) * D // world, dim, [H * D // world, Hkv * D // world, Hkv * D // world]),
                 ("wo", "row", dim, dim // world, None),
                 ("w13", "column", 2 * ffn // world, dim, [ffn // world, ffn // world]),
                 ("w2", "row", dim, ffn // world, None)]
        for si, (name, kind, n, k, segs) in enumerate(specs):
            w = tern(n, k, args.seed + 100003 * rank + 101 * li + si)
            cv, tg, tm, bm = compress_weight(w)
            wbytes += compressed_nbytes(cv, tg, tm, bm)
            dic[name + ".weight_compressed_val"], dic[name + ".weight_TileOffsets_global"] = cv, tg
            dic[name + ".weight_TileOffsets_median"], dic[name + ".weight_bitmap"] = tm, bm
            ws = torch.zeros(4, device=device)
            ws[:len(segs) if segs else 1] = torch.tensor([0.02, 0.03, 0.025][:len(segs) if segs else 1], device=device)
            dic[name + ".weight_scale"] = ws.to(torch.bfloat16)
            if segs:
                dic[name + ".weight_segments"] = torch.tensor(segs)
            if li == 0 and rank == 0:
                dense0[name] = (w.cpu().numpy(), [dic[name + sfx] for sfx in (".weight_compressed_val", ".weight_TileOffsets_global",
                                                                           ".weight_TileOffsets_median", ".weight_bitmap")],
                                dic[name + ".weight_scale"], segs)
            del w
        ones_d = torch.ones(dim // world, device=device)
        ones_f = torch.ones(ffn // world, device=device)
        layers.append((tp.ColumnParallelSpBitLinear(dim, specs[0][2], dic, "wqkv"),
                       tp.RowParallelSpBitLinear(dim // world, dim, dic, "wo", None, ones_d, 1e-5, mode, max_tokens=M),
                       tp.ColumnParallelSpBitLinear(dim, specs[2][2], dic, "w13"),
                       tp.RowParallelSpBitLinear(ffn // world, dim, dic, "w2", None, ones_f, 1e-5, mode,
                                                 gated=True, max_tokens=M)))
    gen.manual_seed(args.seed)
    x0 = torch.randn((M, dim), generator=gen, device=device).to(torch.bfloat16)
    attn = torch.randn((M, dim // world), generator=gen, device=device).to(torch.bfloat16)
    if world > 1:
        dist.broadcast(x0, 0)

    # Sanity check outside the timed region (rank 0, layer 0): every shard's packed weight and the
    # kernels that multiply it, against the CPU oracle - int32 accumulators of all four linears
    # bit-exact, and the column-parallel QKV (explicit scale segments) bf16-identical.
    if rank == 0:
        sys.path.insert(0, os.path.join(ROOT, "oracle"))
        import ternaspmm_oracle as o
        import c_oracle
        c_oracle.load().oracle_set_num_threads(max(1, (os.cpu_count() or 1) // world))   # torchrun exports OMP_NUM_THREADS=1
        one = np.full(M, 0x3F80, np.uint16)
        for name, (wd, packed, ws, segs) in dense0.items():
            n, k = wd.shape
            xq = torch.randint(-128, 128, (M, k), dtype=torch.int8, device=device)
            got = tp._accumulate_i32(xq, packed, n).cpu().numpy()
            acc, _ = c_oracle.ternaspmm(xq.cpu().numpy(), wd, one, np.full(4, 0x3F80, np.uint16), 1)
            if not (got == acc).all():
                raise SystemExit(f"tp bench sanity check failed: int32 accumulators of {name} differ from the oracle")
        wd, packed, ws, segs = dense0["wqkv"]
        xq, s = tp._quant_fused(x0)
        bounds = [sum(segs[:i + 1]) for i in range(2)]
        got = tp._linear_segments(xq, s, packed, ws, bounds, wd.shape[0]).view(torch.int16).cpu().numpy().view(np.uint16)
        acc = o.gemm_i32(xq.cpu().numpy(), wd) if wd.size < (1 << 26) else \
            c_oracle.ternaspmm(xq.cpu().numpy(), wd, one, np.full(4, 0x3F80, np.uint16), 1)[0]
        g = (np.arange(wd.shape[0]) >= bounds[0]).astype(np.int64) + (np.arange(wd.shape[0]) >= bounds[1])
        v = (acc.astype(np.float32) / s.float().cpu().numpy().reshape(-1, 1)).astype(np.float32) * \
            ws.float().cpu().numpy()[g][None, :]
        if not (got == o.f32_to_bf16_bits(v)).all():
            raise SystemExit("tp bench sanity check failed: sharded QKV output differs from the oracle")
    dense0.clear()
    # rank 0 has just spent seconds on the host-side check: meet here, or the other ranks' first fused
    # calls would wait for it on the device beyond the library's bounded-wait limit
    env.barrier()

    def step():
        x = x0
        for qkv, wo, w13, w2 in layers:
            qkv(x)
            h = wo(attn, residual=x)
            x = w2(w13(h), residual=h)
        return x

    class _Eager:
        def replay(self):
            step()

    with torch.cuda.stream(env.stream):
        for _ in range(2):
            step()
        env.stream.synchronize()
        if args.no_graph:
            graph = _Eager()
        else:
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph, stream=env.stream):
                y = step()
    ms = env.time_replays(graph.replay, args.steps, args.warmup, min_load_s=0.3)
    tp.check_status()     # a device-side wait that ran out would have poisoned the outputs
    if not torch.isfinite(step().float()).all():
        raise SystemExit("tp bench: non-finite outputs")
    wb = torch.tensor([float(wbytes)], dtype=torch.float64, device=device)
    if world > 1:
        dist.all_reduce(wb)
    peak, kind = measured_peak()
    val = float(wb.item()) * args.steps / (ms * 1e-3) / 1e9
    res = {"mode": mode, "ms_per_step": ms / args.steps, "layers": L, "tokens": M, "tp": world,
           "compressed_weight_GBps": val, "per_gpu_frac": val / world / peak, "peak_kind": "of " + kind,
           "collective": {"single": "one NCCL all-reduce per row-parallel linear",
                          "fused": "reduce-scatter + all-gather inside the finish kernel over peer memory (plain NVLink "
                                   "loads and stores)",
                          "exact": "three all-reduces per row-parallel linear (bit-exact mode)"}[mode],
           "gpu_launches": (6 if mode == "exact" else 10) * L * args.steps}
    del layers, graph
    torch.cuda.empty_cache()
    return res


def run_tp_arm(args):
    env = Env()
    M = args.tokens if args.tokens != 8 else 64
    L = args.layers if args.layers != 30 else 4
    sampler = ClockSampler(env.local_rank)
    if env.rank == 0:
        sampler.start()
    res = tp_stack(env, args, args.tp_mode, M, L)
    clocks = sampler.stop() if env.rank == 0 else None
    if env.rank == 0:
        peak, kind = measured_peak()
        line = {"metric": "ternaspmm_tp_compressed_weight_GBps", "value": res["compressed_weight_GBps"], "unit": "GB/s",
                "n_gpus": env.world, "steps": args.steps, "warmup": args.warmup, "ms_per_step": res["ms_per_step"],
                "higher_is_better": True, "scaling": "strong", "vs_baseline": None,
                "dtype": "int8xternary->int32->bf16", "data": "synthetic",
                "config": {"workload": f"tp_linear_stack_8192x28672_bs{M}", "layers": L, "tokens": M, "tp": env.world,
                           "row_parallel_mode": args.tp_mode, "collective": res["collective"],
                           "l2_policy": "inputs larger than L2: every step streams all layers' weight shards"},
                "roofline": {"bound": "hbm", "achieved": res["compressed_weight_GBps"] / env.world, "peak": peak,
                             "unit": "GB/s", "frac": res["per_gpu_frac"], "peak_kind": "of " + kind, "traffic": None,
                             "note": "per-GPU compressed-weight bytes per second"},
                "gpu_launches": res["gpu_launches"], "clocks": clocks}
        print(json.dumps(line), flush=True)
    _finish(env.world)


# ----------------------------------------------------------------------------
# End-to-end decode arm: the 30-layer BitNet-2B architecture
# with random-init ternary weights and a dense bf16 tied embedding / head, prompt
# of seeded random ids, greedy generation; value = decode tokens per second.
# ----------------------------------------------------------------------------

def cpu_decode_sample(bsz, layers, seconds_budget=10.0, seed=1234):
    """PyTorch-CPU model path of one decode step, timed on the host cores: one decoder layer of the
    BitNet-2B architecture as the reference's dense comparator computes it (quant_input, F.linear on
    the de-quantised ternary weight, division by the scale; RMSNorm and sub-layer norms, RoPE,
    attention over a 640-token bf16 cache, relu^2 gate) plus the tied output head, all float32
    torch CPU ops.  A step costs `layers` x the layer time + the head time; returns tokens/s."""
    import torch
    import torch.nn.functional as F
    torch.manual_seed(seed)
    dim, H, Hkv, D, ffn, vocab, L = 2560, 20, 5, 128, 6912, 128256, 640
    torch.set_num_threads(os.cpu_count() or 1)    # launchers export OMP_NUM_THREADS=1; use the host's cores
    cores = torch.get_num_threads()

    def tern(n, k):
        r = torch.rand(n, k)
        return torch.where(r < P_ZERO, torch.zeros(()), torch.where(torch.rand(n, k) < 0.5, -torch.ones(()), torch.ones(())))

    wqkv, wo, w13, w2 = tern((H + 2 * Hkv) * D, dim), tern(dim, dim), tern(2 * ffn, dim), tern(dim, ffn)
    head = torch.randn(vocab, dim) * 0.02
    ck, cv = torch.randn(bsz, Hkv, L, D), torch.randn(bsz, Hkv, L, D)
    g = [torch.ones(dim), torch.ones(dim), torch.ones(dim), torch.ones(ffn)]

    def norm(x, w):
        return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + 1e-5) * w

    def lin(x, w):
        s = 127 / x.abs().max(-1, keepdim=True).values.clamp(min=1e-5)
        return F.linear((x * s).round().clamp(-128, 127), w) / s * 0.02

    def layer(x):
        qkv = lin(norm(x, g[0]), wqkv)
        q = qkv[:, : H * D].view(bsz, 1, H, D).transpose(1, 2)
        k = qkv[:, H * D: (H + Hkv) * D].view(bsz, Hkv, 1, D)
        v = qkv[:, (H + Hkv) * D:].view(bsz, Hkv, 1, D)
        ck[:, :, L - 1: L], cv[:, :, L - 1: L] = k, v
        o = F.scaled_dot_product_attention(q, ck.repeat_interleave(H // Hkv, 1), cv.repeat_interleave(H // Hkv, 1))
        h = x + lin(norm(o.transpose(1, 2).reshape(bsz, H * D), g[1]), wo)
        x13 = lin(norm(h, g[2]), w13)
        inner = torch.relu(x13[:, :ffn]) ** 2 * x13[:, ffn:]
        return h + lin(norm(inner, g[3]), w2)

    x = torch.randn(bsz, dim)
    with torch.inference_mode():
        layer(x), F.linear(x, head)
        t0 = time.perf_counter()
        layer(x)
        one = time.perf_counter() - t0
        reps = max(2, min(200, int(0.7 * seconds_budget / max(one, 1e-6))))
        t0 = time.perf_counter()
        for _ in range(reps):
            x = layer(x)
        t_layer = (time.perf_counter() - t0) / reps
        hreps = max(2, min(50, int(0.3 * seconds_budget / max(one * 4, 1e-6))))
        t0 = time.perf_counter()
        for _ in range(hreps):
            F.linear(x, head)
        t_head = (time.perf_counter() - t0) / hreps
    step = layers * t_layer + t_head
    return bsz / step, cores, f"{reps} passes of one decoder layer and {hreps} of the output head at batch {bsz}, " \
                               f"float32 torch CPU ops; step = {layers} x layer + head"


def decode_run(args, bsz, fused, reps):
    """Greedy generation of 128 tokens after a 512-token prompt at batch `bsz`; best of `reps` runs."""
    import torch
    from ternainfer_b200.generate import FastGen, GenArgs, build_random_model
    from ternainfer_b200.model import ModelArgs
    margs = ModelArgs(n_layers=args.layers, fused_glue=fused)
    model, _ = build_random_model(margs, 512 + 128, args.seed)
    gen = FastGen(model, GenArgs(128, bsz, 512, True))
    g = torch.Generator(device="cuda").manual_seed(args.seed + 1)
    prompt = torch.randint(0, margs.vocab_size, (bsz, 512), generator=g, device="cuda")
    gen.generate(prompt)            # captures the graphs
    best, first = None, None
    for _ in range(reps):
        toks, st = gen.generate(prompt)
        first = toks[0, :8].tolist()
        if best is None or st["decode_tokens_per_s"] > best["decode_tokens_per_s"]:
            best = st
    del gen, model
    torch.cuda.empty_cache()
    return best, first


def decode_leg(args):
    """Decode tokens/s of the 30-layer model (prompt 512, 128 generated tokens) at batch 1 and 8, with
    the fused front-ends and with plain torch glue between the linears, plus the PyTorch-CPU decode step."""
    out = {"layers": args.layers, "prompt": 512, "generate": 128,
           "note": "random-init weights give near-tied logits over 128256 words, so the two glue variants (another "
                   "fp32 summation order in RMSNorm, another attention kernel) choose different tokens; with the norm's "
                   "summation order held equal the fused path returns the eager model's logits and tokens exactly "
                   "(tests/test_gpu_model.py, 30 layers, batch 1 and 8)"}
    for bsz in (1, 8):
        entry = {}
        for fused in (True, False):
            st, first = decode_run(args, bsz, fused, 2)
            entry["fused_glue" if fused else "torch_glue"] = {
                "decode_tokens_per_s": st["decode_tokens_per_s"], "prefill_tokens_per_s": st["prefill_tokens_per_s"],
                "first_tokens": first}
        cpu_tps, cores, sample = cpu_decode_sample(bsz, args.layers, seconds_budget=6.0)
        entry["cpu_baseline"] = {"value": cpu_tps, "unit": "tokens/s", "cores": cores, "kind": "port", "sample": sample}
        out[f"bs{bsz}"] = entry
    return out


def run_decode_arm(args):
    import torch
    torch.cuda.set_device(0)
    bsz = args.tokens if args.tokens in (1, 8) else 1
    sampler = ClockSampler(0)
    sampler.start()
    best, _ = decode_run(args, bsz, not args.unfused, max(1, args.steps // 10))
    clocks = sampler.stop()
    line = {"metric": "decode_tokens_per_s", "value": best["decode_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": 1e3 * bsz / best["decode_tokens_per_s"],
            "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "int8xternary->int32->bf16",
            "data": "synthetic",
            "config": {"workload": f"bitnet2b_greedy_decode_bs{bsz}", "layers": args.layers, "prompt": 512,
                       "generate": 128, "fused_glue": not args.unfused, "seed": args.seed,
                       "prefill_tokens_per_s": best["prefill_tokens_per_s"]},
            "clocks": clocks}
    cpu_tps, cores, sample = cpu_decode_sample(bsz, args.layers)
    line["cpu_baseline"] = {"value": cpu_tps, "unit": "tokens/s", "cores": cores, "kind": "port", "sample": sample}
    print(json.dumps(line), flush=True)


# ----------------------------------------------------------------------------
# Kepovik workload: the decoder of ternainfer_b200/kepovik.py beside the ternary
# model of equal width, feed-forward, heads and layer count (the closest one the
# framework has), whole models and kernel by kernel.
# ----------------------------------------------------------------------------

KEPOVIK_SIZES = {   # width, feed-forward, attention heads, kv heads, head dim, delta heads, delta dim, layers
    "2560": (2560, 6912, 20, 5, 128, 40, 64, 30),
    "4096": (4096, 14336, 32, 8, 128, 64, 64, 8),
}
KEPOVIK_VOCAB, KEPOVIK_CHUNK, KEPOVIK_RANK, KEPOVIK_STREAMS = 128256, 2048, 64, 4


def kepovik_config(size):
    """Delta and attention layers in turn, a feed-forward in every layer."""
    width, ff, heads, kv, dim, dh, dd, layers = KEPOVIK_SIZES[size]
    mlp = {"kind": "dense", "ff": ff}
    delta = {"type": "general_delta", "mixer": {"heads": dh, "dim": dd}, "mlp": mlp}
    attn = {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim,
                                                       "mask": {"size": KEPOVIK_CHUNK}, "scale": dim ** -0.5}}
    return {"architecture": "Kepovik", "vocab": KEPOVIK_VOCAB, "width": width, "streams": KEPOVIK_STREAMS, "norm": {"eps": 1e-5},
            "residual_mult": 0.5, "layers": [delta if i % 2 == 0 else attn for i in range(layers)],
            "embedding": {"bigram": {"buckets": 65521, "mul_prev": 31, "mul_cur": 17}}}


def kepovik_model(size, max_len, seed):
    import torch
    from ternainfer_b200.kepovik import Kepovik, parse_config, random_checkpoint
    args = parse_config(kepovik_config(size))
    return Kepovik(args, random_checkpoint(args, KEPOVIK_RANK, seed), max_seq_len=max_len, dtype=torch.bfloat16).cuda()


def ternary_model(size, max_len, seed):
    from ternainfer_b200.generate import build_random_model
    from ternainfer_b200.linear import reserve_workspace
    from ternainfer_b200.model import ModelArgs
    width, ff, heads, kv, dim, _, _, layers = KEPOVIK_SIZES[size]
    reserve_workspace(2 * ff * width)
    return build_random_model(ModelArgs(dim=width, n_layers=layers, n_heads=heads, n_kv_heads=kv, ffn_dim=ff,
                                        vocab_size=KEPOVIK_VOCAB, fused_glue=True), max_len, seed)[0]


def graph_us(torch, calls, steps, warmup):
    """Device time per call of a list of calls captured in one graph (CUDA events, `steps` replays)."""
    with torch.inference_mode():
        for c in calls:
            c()
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            for c in calls:
                c()
        for _ in range(warmup):
            g.replay()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        for _ in range(steps):
            g.replay()
        b.record()
        torch.cuda.synchronize()
    return a.elapsed_time(b) * 1e3 / (steps * len(calls))


def model_speed(torch, build, size, args):
    """Prompt and decode tokens/s of a model through FastGen's captured graphs."""
    from ternainfer_b200.generate import FastGen, GenArgs
    out = {}
    for P, B in ((512, 1), (2048, 1), (512, 8)):
        model = build(size, P + 128, args.seed)
        gen = FastGen(model, GenArgs(128, B, P, True))
        g = torch.Generator(device="cuda").manual_seed(args.seed + 1)
        gen.generate(torch.randint(0, KEPOVIK_VOCAB, (B, P), generator=g, device="cuda"))
        gen._pos.fill_(P + 64)
        ev = [torch.cuda.Event(enable_timing=True) for _ in range(3)]
        n_pre, n_dec = max(3, args.steps // 10), args.steps
        for _ in range(args.warmup):
            gen._prefill_graph.replay()
            gen._decode_graph.replay()
        torch.cuda.synchronize()
        ev[0].record()
        for _ in range(n_pre):
            gen._prefill_graph.replay()
        ev[1].record()
        for _ in range(n_dec):
            gen._decode_graph.replay()
        ev[2].record()
        torch.cuda.synchronize()
        pre, dec = ev[0].elapsed_time(ev[1]) / n_pre, ev[1].elapsed_time(ev[2]) / n_dec
        out[f"prompt{P}_batch{B}"] = {"prefill_ms": pre, "prefill_tokens_per_s": 1e3 * P * B / pre, "decode_ms": dec,
                                      "decode_tokens_per_s": 1e3 * B / dec}
        del gen, model
        torch.cuda.empty_cache()
    return out


def kernel_table(torch, out, args):
    """put(model, name, calls, bytes, flops): times the calls and files microseconds, algorithmic bytes and matrix FLOPs, and
    the fraction of the larger of the two bounds under out[model][name]."""
    peak, tf = out["peaks"]["hbm_gbs"], out["peaks"]["bf16_tflops"]

    def put(model, name, calls, nbytes, flops=0.0):
        us = graph_us(torch, calls, max(5, args.steps // 5), args.warmup)
        bound = max(nbytes / peak / 1e3, flops / tf / 1e6)
        out[model][name] = {"us": us, "bytes": nbytes, "flops": flops, "bound_us": bound, "frac": bound / us}
        torch.cuda.empty_cache()
    return put


def copies(nbytes):
    """Copies of an operand that together are larger than the L2."""
    return max(2, min(400, int(160e6 / nbytes) + 1))


def measured_tflops():
    try:
        return float(json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json")))["bf16_tflops"])
    except Exception:
        return 1590.0


def kepovik_kernels(torch, size, args):
    """Every kernel of both models at this size: microseconds, algorithmic bytes and matrix FLOPs, and the fraction of the
    larger of the two bounds (measured copy rate, measured bf16 GEMM rate; the int8 GEMM against the latter too)."""
    from ternainfer_b200 import decoder_ops as ops
    from ternainfer_b200.linear import lm_head_argmax, rmsnorm_quant
    width, ff, heads, kv, dim, dh, dd, _ = KEPOVIK_SIZES[size]
    peak, kind = measured_peak()
    tf = measured_tflops()
    S, V, bf, dev = KEPOVIK_STREAMS, KEPOVIK_VOCAB, torch.bfloat16, "cuda"
    g = torch.Generator(device=dev).manual_seed(args.seed)
    rnd = lambda *shape, dtype=bf, scale=1.0: (scale * torch.randn(shape, generator=g, device=dev)).to(dtype)
    out = {"peaks": {"hbm_gbs": peak, "bf16_tflops": tf, "kind": kind}, "kepovik": {}, "ternary": {}}
    put = kernel_table(torch, out, args)

    nd, na = 5 * dh * dd + KEPOVIK_RANK, 2 * heads * dim + 2 * kv * dim
    off_d = {n: i * dh * dd for i, n in enumerate(("r", "k", "v", "a", "g", "w1"))}
    off_a = {"q": 0, "k": heads * dim, "v": (heads + kv) * dim, "g": (heads + 2 * kv) * dim}
    f32 = lambda *shape: rnd(*shape, dtype=torch.float32, scale=0.3)
    for B in (1, 8):
        tag, at = f"decode_batch{B}", torch.tensor([KEPOVIK_CHUNK - 1], device=dev)
        for name, N, K, relu2 in (("delta_in", nd, width, False), ("mixer_out", width, dh * dd, False), ("attn_in", na, width, False),
                                  ("ff_up_relu2", ff, width, True), ("ff_down", width, ff, False)):
            nb = 2.0 * (N * K + B * (N + K))
            x, ws = rnd(B, K), [rnd(N, K, scale=K ** -0.5) for _ in range(copies(nb))]
            put("kepovik", f"{tag}/linear_{name}", [lambda w=w: ops.linear(x, w, relu2=relu2, step=True) for w in ws], nb, 2.0 * B * N * K)
            del ws
        xs, y, h1, w1 = rnd(B, S, width, dtype=torch.float32), rnd(B, width), f32(S), f32(width)
        mix = torch.eye(S, device=dev)
        put("kepovik", f"{tag}/streams_norm", [lambda: ops.hyper_norm(xs, w1, 1e-5, bf, w_in=h1, weight_offset=1.0, y=y, mix=mix, w_out=h1,
                                                                      step=True)] * 20, B * width * (8.0 * S + 4))
        nb = B * dh * dd * dd * 8.0 + 2.0 * dh * dd * KEPOVIK_RANK + 12.0 * B * dh * dd
        st = [torch.zeros((B, dh, dd, dd), device=dev) for _ in range(copies(nb))]
        z, w2, v1 = rnd(B, nd), rnd(dh * dd, KEPOVIK_RANK, scale=0.1), f32(dh * dd)
        put("kepovik", f"{tag}/delta_step", [lambda s=s: ops.delta_rule(z, off_d, w2, v1, v1, v1, s, at, 1, 1e-5, step=True) for s in st], nb)
        del st
        nb = 4.0 * B * kv * KEPOVIK_CHUNK * dim
        cc = [(rnd(B, kv, KEPOVIK_CHUNK, dim), rnd(B, kv, KEPOVIK_CHUNK, dim)) for _ in range(copies(nb))]
        z, qn, hb = rnd(B, na), f32(dim), f32(heads) - 4
        put("kepovik", f"{tag}/attention_2048", [lambda c=c: ops.sigmoid_attention(z, off_a, qn, qn, hb, hb, c, at, 1, heads, KEPOVIK_CHUNK,
                                                                                   dim ** -0.5, 1e-5, step=True) for c in cc], nb)
        del cc
        hd, W = rnd(B, width), rnd(V, width, scale=width ** -0.5)
        put("kepovik", f"{tag}/output_head", [lambda: ops.output_argmax(hd, W)], 2.0 * V * width)
        del W
    T = 2048
    pos = torch.arange(T, device=dev)
    xs = [rnd(T, S, width, dtype=torch.float32) for _ in range(3)]
    y = rnd(T, width)
    put("kepovik", "prefill2048/streams_norm", [lambda x=x: ops.hyper_norm(x, w1, 1e-5, bf, w_in=h1, weight_offset=1.0, y=y, mix=mix, w_out=h1)
                                               for x in xs], T * width * (8.0 * S + 4))
    del xs
    zs, state = [rnd(T, nd) for _ in range(3)], torch.zeros((1, dh, dd, dd), device=dev)
    put("kepovik", "prefill2048/delta_rule", [lambda z=z: ops.delta_rule(z, off_d, w2, v1, v1, v1, state, pos, T, 1e-5) for z in zs],
        2.0 * T * (nd + dh * dd))
    out["kepovik"]["prefill2048/delta_rule"]["fp32_fma"] = 5.0 * T * dh * dd * dd
    zs, cc = [rnd(T, na) for _ in range(5)], (rnd(1, kv, T, dim), rnd(1, kv, T, dim))
    att = 2.0 * T * (T + 1) * heads * dim
    put("kepovik", "prefill2048/attention", [lambda z=z: ops.sigmoid_attention(z, off_a, qn, qn, hb, hb, cc, pos, T, heads, KEPOVIK_CHUNK,
                                                                               dim ** -0.5, 1e-5) for z in zs], 2.0 * T * (na + heads * dim), att)
    x, ws = rnd(T, width), [rnd(ff, width, scale=width ** -0.5) for _ in range(copies(2.0 * ff * width))]
    put("kepovik", "prefill2048/linear_ff_up_relu2", [lambda w=w: ops.linear(x, w, relu2=True) for w in ws],
        2.0 * (T * (width + ff) + ff * width), 2.0 * T * ff * width)
    put("kepovik", "prefill2048/linear_ff_up", [lambda w=w: ops.linear(x, w) for w in ws], 2.0 * (T * (width + ff) + ff * width),
        2.0 * T * ff * width)
    del zs, ws

    # the ternary model's kernels
    model = ternary_model(size, T, args.seed)
    from flash_attn import flash_attn_with_kvcache
    L, lay = model.layers, list(model.layers)
    comp = lambda m: sum(t.numel() * t.element_size() for t in (m.weight_compressed_val, m.weight_TileOffsets_global,
                                                                m.weight_TileOffsets_median, m.weight_bitmap))
    qkv = (heads + 2 * kv) * dim
    for B, tag in ((1, "decode_batch1"), (8, "decode_batch8"), (T, "prefill2048")):
        for name, pick in (("wqkv", lambda l: l.attention.wqkv), ("wo", lambda l: l.attention.wo), ("w13", lambda l: l.feed_forward.w13),
                           ("w2", lambda l: l.feed_forward.w2)):
            N, K = pick(L[0]).out_features, pick(L[0]).in_features
            xq, sc = torch.randint(-127, 128, (B, K), dtype=torch.int8, device=dev), torch.ones((B, 1), dtype=bf, device=dev)
            put("ternary", f"{tag}/linear_{name}", [lambda l=l: pick(l).forward_quantized(xq, sc) for l in lay],
                comp(pick(L[0])) + B * (K + 2.0 * N), 2.0 * B * N * K)
        x = rnd(B, width)
        nw = rnd(width)
        put("ternary", f"{tag}/norm_quant", [lambda: rmsnorm_quant(x, nw, 1e-5)] * 10, 3.0 * B * width)
        nb_b, t_q = (B, 1) if B <= 8 else (1, B)
        q = [rnd(nb_b, t_q, heads, dim) for _ in range(3)]
        k1 = rnd(nb_b, t_q, kv, dim)
        nb = 4.0 * nb_b * kv * T * dim
        cc = [(rnd(nb_b, T, kv, dim), rnd(nb_b, T, kv, dim)) for _ in range(copies(nb))]
        seen = torch.full((nb_b,), T - t_q, dtype=torch.int32, device=dev)
        tabs = rnd(T, dim // 2)
        put("ternary", f"{tag}/attention_2048", [lambda i=i, c=c: flash_attn_with_kvcache(
            q[i % 3], c[0], c[1], k=k1, v=k1, rotary_cos=tabs, rotary_sin=tabs, cache_seqlens=seen, causal=True, rotary_interleaved=True)
            for i, c in enumerate(cc[:60])], nb if t_q == 1 else 2.0 * T * (qkv + heads * dim), 0.0 if t_q == 1 else att)
        del cc, q
        if B <= 8:
            hd = rnd(B, width)
            put("ternary", f"{tag}/output_head", [lambda: lm_head_argmax(hd, model.tok_embeddings.weight, False, True)], 2.0 * V * width)
    return out


def run_kepovik_arm(args):
    import torch
    torch.cuda.set_device(0)
    sampler = ClockSampler(0)
    sampler.start()
    res = {}
    for size in KEPOVIK_SIZES:
        res[size] = {"layers": KEPOVIK_SIZES[size][-1], "kepovik": model_speed(torch, kepovik_model, size, args),
                     "ternary": model_speed(torch, ternary_model, size, args), "kernels": kepovik_kernels(torch, size, args)}
    clocks = sampler.stop()
    best = res["2560"]["kepovik"]["prompt512_batch1"]
    line = {"metric": "kepovik_decode_tokens_per_s", "value": best["decode_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": best["decode_ms"], "higher_is_better": True, "scaling": "weak",
            "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
            "config": {"workload": "kepovik_2560_30_layers_prompt512_batch1", "vocab": KEPOVIK_VOCAB, "chunk": KEPOVIK_CHUNK,
                       "decay_rank": KEPOVIK_RANK, "streams": KEPOVIK_STREAMS, "seed": args.seed,
                       "l2_policy": "weights, states and caches larger than L2 in rotation; decode activations stay in L2"},
            "sizes": res, "clocks": clocks}
    print(json.dumps(line), flush=True)


# ----------------------------------------------------------------------------
# Sidirax workload: the decoder of ternainfer_b200/sidirax.py beside Kepovik of equal
# width, layers, heads and active feed-forward width (the closest model: recurrent and
# attention layers with dense bf16 weights), whole models and kernel by kernel.
# ----------------------------------------------------------------------------

SIDIRAX_EXPERTS, SIDIRAX_TOP, SIDIRAX_ROT, SIDIRAX_KV_RANK = 32, 4, 64, 512


def sidirax_config(size):
    """wkv and latent attention layers in turn, every second attention layer on the latent of the one before; the first
    feed-forward dense, the others experts whose chosen ones together are as wide."""
    width, ff, heads, _, dim, wh, wd, layers = KEPOVIK_SIZES[size]
    rot = {"base": 10000.0, "dims": SIDIRAX_ROT, "scaling": {"factor": 4.0, "original": 1024, "fast": 32.0, "slow": 1.0}}
    out = []
    for i in range(layers):
        mlp = {"kind": "dense", "ff": ff, "limit": 7.0} if i == 0 else \
            {"kind": "moe", "expert": {"ff": ff // SIDIRAX_TOP}, "router": {"experts": SIDIRAX_EXPERTS, "top": SIDIRAX_TOP}}
        if i % 2 == 0:
            out.append({"type": "wkv", "mixer": {"heads": wh, "dim": wd}, "mlp": mlp})
            continue
        mixer = {"heads": heads, "dim": dim, "rot_dim": SIDIRAX_ROT, "vdim": dim, "q_rank": width // 2, "kv_rank": SIDIRAX_KV_RANK,
                 "scale": (dim + SIDIRAX_ROT) ** -0.5, "rot": rot}
        if i % 4 == 3:
            mixer["kv_from"] = i - 2
        out.append({"type": "latent_attention", "mixer": mixer, "mlp": mlp})
    return {"architecture": "Sidirax", "vocab": KEPOVIK_VOCAB, "width": width, "norm": {"eps": 1e-5}, "layers": out}


def sidirax_model(size, max_len, seed):
    import torch
    from ternainfer_b200.sidirax import Sidirax, parse_config, random_checkpoint
    args = parse_config(sidirax_config(size))
    return Sidirax(args, random_checkpoint(args, KEPOVIK_RANK, seed), max_seq_len=max_len, dtype=torch.bfloat16).cuda()


def sidirax_kernels(torch, size, args):
    """Every kernel of the model at this size; bytes count every weight that is used once (for experts: the distinct chosen
    ones), every cache entry and every activation once."""
    from ternainfer_b200 import decoder_ops as ops
    width, ff, heads, _, dim, wh, wd, _ = KEPOVIK_SIZES[size]
    peak, kind = measured_peak()
    out = {"peaks": {"hbm_gbs": peak, "bf16_tflops": measured_tflops(), "kind": kind}, "sidirax": {}}
    table = kernel_table(torch, out, args)
    put = lambda name, calls, nbytes, flops=0.0: table("sidirax", name, calls, nbytes, flops)
    bf, dev, eps = torch.bfloat16, "cuda", 1e-5
    g = torch.Generator(device=dev).manual_seed(args.seed)
    rnd = lambda *shape, dtype=bf, scale=1.0: (scale * torch.randn(shape, generator=g, device=dev)).to(dtype)
    f32 = lambda *shape, scale=0.3: rnd(*shape, dtype=torch.float32, scale=scale)
    E, top, rot, R, V, n = SIDIRAX_EXPERTS, SIDIRAX_TOP, SIDIRAX_ROT, SIDIRAX_KV_RANK, KEPOVIK_VOCAB, wh * wd
    fe, qr, dq, ld, rank, S = ff // top, width // 2, dim + rot, R + rot, KEPOVIK_RANK, 2048
    trig, w1, mu, silu = f32(S, rot), f32(width), f32(5, width), ops.silu_gate()
    clamp = ops.clamped_gate(1.702, 7.0)
    uk, uv, sink = rnd(heads * dim, R, scale=R ** -0.5), rnd(heads * dim, R, scale=R ** -0.5), f32(heads)
    uk_t = uk.view(heads, dim, R).transpose(1, 2).contiguous()
    w2, w0, u, nw = rnd(n, rank, scale=0.1), f32(n) - 3, f32(wh, wd), f32(n)
    rw, rb = rnd(E, width, scale=width ** -0.5), f32(E)
    up = [rnd(E, 2 * fe, width, scale=width ** -0.5) for _ in range(2)]
    down = [rnd(E, width, fe, scale=fe ** -0.5) for _ in range(2)]
    wo = [rnd(width, n, scale=n ** -0.5) for _ in range(8)]
    for B in (1, 8):
        tag, at = f"decode_batch{B}", torch.tensor([S - 1], device=dev)
        for name, N, K in (("latent_in", qr + R + rot, width), ("latent_uq", heads * dq, qr)):
            nb = 2.0 * (N * K + B * (N + K))
            x, ws = rnd(B, K), [rnd(N, K, scale=K ** -0.5) for _ in range(copies(nb))]
            put(f"{tag}/linear_{name}", [lambda w=w: ops.linear(x, w, step=True) for w in ws], nb, 2.0 * B * N * K)
        N = 4 * n + rank
        nb = 2.0 * (N * width + B * (N + 5 * width))
        x, ws = rnd(5, B, width), [rnd(N, width, scale=width ** -0.5) for _ in range(copies(nb))]
        put(f"{tag}/linear_wkv_in", [lambda w=w: ops.rows_linear(x, w, seg_rows=n, step=True) for w in ws], nb, 2.0 * B * N * width)
        nb = 2.0 * (2 * ff * width + B * (ff + width))
        x, ws, bias = rnd(B, width), [rnd(2 * ff, width, scale=width ** -0.5) for _ in range(copies(nb))], f32(2 * ff)
        put(f"{tag}/dense_up_clamped", [lambda w=w: ops.rows_linear(x, w, bias, clamp, step=True) for w in ws], nb, 4.0 * B * ff * width)
        nb = 2.0 * (ff * width + width * n + B * (ff + n + width))
        act, a, ws, db = rnd(B, ff), rnd(B, n), [rnd(width, ff, scale=ff ** -0.5) for _ in range(copies(nb))], f32(width)
        put(f"{tag}/dense_down_and_mixer_out", [lambda w=w, o=wo[i % 8]: ops.down_step(act, w, db, rest=a, w_rest=o, step=True) for i, w in enumerate(ws)],
            nb, 2.0 * B * (ff + n) * width)
        del ws
        routes, acts = [ops.Routing(rnd(B, width), rw, rb, top) for _ in range(20)], []
        tickets = torch.zeros(20, dtype=torch.int32, device=dev)           # zeroed once per list; in the model, by the projection before
        for i, r in enumerate(routes):
            r.logits.copy_(ops.linear_fp32(r.x, rw))
            r.ticket = tickets[i:i + 1]
            acts.append(ops.expert_step(r, up[0], silu))
        used = sum(r.chosen.unique().numel() for r in routes) / 20
        put(f"{tag}/routing_and_expert_up", [lambda i=i, r=r: (tickets.zero_() if i == 0 else None, ops.expert_step(r, up[i % 2], silu, True))
                                             for i, r in enumerate(routes)],
            2.0 * (used * 2 * fe * width + B * (width + top * fe)), 4.0 * B * top * fe * width)
        put(f"{tag}/expert_down_and_mixer_out", [lambda t=t, r=r, w=down[i % 2], o=wo[i % 8]: ops.down_step(t, w, None, r, a, o, True)
                                                 for i, (t, r) in enumerate(zip(acts, routes))],
            2.0 * (used * fe * width + width * n + B * (top * fe + n + width)), 2.0 * B * (top * fe + n) * width)
        xr, y, prev = f32(B, 1, width), rnd(B, width), rnd(B, width)
        put(f"{tag}/residual_norm", [lambda: ops.hyper_norm(xr, w1, eps, bf, y=y, step=True)] * 20, 12.0 * B * width)
        put(f"{tag}/residual_norm_shift", [lambda: ops.hyper_norm(xr, w1, eps, bf, y=y, shift=(mu, prev, at), step=True)] * 20, B * width * 26.0 + 20.0 * width)
        nb = B * wh * wd * wd * 8.0 + 2.0 * n * rank + 12.0 * B * n
        st, z = [torch.zeros((B, wh, wd, wd), device=dev) for _ in range(copies(nb))], rnd(B, 4 * n + rank)
        r, k, v, gt, t1 = (z[:, i * n:] for i in range(5))
        put(f"{tag}/wkv_step", [lambda s=s: ops.wkv(r, k, v, gt, t1, w2, w0, u, nw, s, at, 1, eps, True) for s in st], nb)
        del st
        nb = 2.0 * B * S * ld + 4.0 * heads * dim * R
        cc = [rnd(B, S, ld) for _ in range(copies(2.0 * B * S * ld))]
        z, q, qn, kn = rnd(B, qr + ld), rnd(B, heads * dq), f32(qr), f32(R)
        qa = ops.absorb(q, uk, uk_t, heads, dim, rot, R, ld, trig, at, 1)
        put(f"{tag}/latent_norms_append", [lambda c=c: ops.latent_prep(z, 0, qn, at, 1, eps, c, qr, kn, R, rot, trig, True) for c in cc], 4.0 * B * (qr + ld))
        put(f"{tag}/latent_absorb", [lambda: ops.absorb(q, uk, uk_t, heads, dim, rot, R, ld, trig, at, 1, True)] * 20, 2.0 * (heads * dim * R + B * heads * (dq + ld)))
        put(f"{tag}/latent_attention_2048", [lambda c=c: ops.latent_attention_step(qa, c, uv, sink, at, 1, dim, 0.07, True) for c in cc],
            2.0 * B * S * ld + 2.0 * heads * dim * R, 2.0 * B * heads * S * (ld + R))
        put(f"{tag}/latent_attention_2048_all", [lambda c=c: ops.latent_attention_step(ops.absorb(q, uk, uk_t, heads, dim, rot, R, ld, trig, at, 1, True), c, uv, sink,
                                                                                       at, 1, dim, 0.07, True) for c in cc], nb, 2.0 * B * heads * S * (ld + R))
        del cc
        hd, W = rnd(B, width), rnd(V, width, scale=width ** -0.5)
        put(f"{tag}/output_head", [lambda: ops.output_argmax(hd, W)], 2.0 * V * width)
        del W
    T, tag = S, "prefill2048"
    pos, h = torch.arange(T, device=dev), rnd(T, width)
    xr, y, ye = [f32(T, 1, width) for _ in range(4)], rnd(T, width), rnd(T * top, width)
    slots, sw = torch.randperm(T * top, device=dev).int().view(T, top), torch.rand((T, top), device=dev)
    put(f"{tag}/residual_norm", [lambda x=x: ops.hyper_norm(x, w1, eps, bf, y=y) for x in xr], T * width * 12.0)
    put(f"{tag}/residual_norm_experts", [lambda x=x: ops.hyper_norm(x, w1, eps, bf, y=y, y2=ye, slots=slots, slot_w=sw) for x in xr], T * width * (12.0 + 2 * top))
    del xr, ye
    prev = rnd(1, width)
    put(f"{tag}/token_shift", [lambda: ops.token_shift(h, mu, prev, pos, T)] * 5, T * width * 12.0)
    zs, state = [rnd(4, T, n) for _ in range(2)], torch.zeros((1, wh, wd, wd), device=dev)
    t1, zw = rnd(T, rank), f32(T, n)
    put(f"{tag}/wkv", [lambda z=z: ops.wkv(z[0], z[1], z[2], z[3], t1, w2, w0, u, nw, state, pos, T, eps, zw=zw) for z in zs], T * n * 14.0)
    out["sidirax"][f"{tag}/wkv"]["fp32_fma"] = 2.0 * T * n * wd
    x5, ws = rnd(4, T, width), [rnd(4, n, width, scale=width ** -0.5) for _ in range(4)]
    put(f"{tag}/linear_wkv_in", [lambda w=w: torch.bmm(x5, w.transpose(1, 2)) for w in ws], 8.0 * (T * (n + width) + n * width), 8.0 * T * n * width)
    del zs, ws, x5
    cache, ukv = rnd(1, T, ld), torch.cat([uk, uv])
    qs = [rnd(T, heads * dq) for _ in range(5)]
    att = T * (T + 1.0) * heads * (dq + dim)
    put(f"{tag}/attention", [lambda q=q: ops.latent_attention_prompt(q, ukv, cache, sink, 0, T, heads, dim, rot, dim, R, 0.07) for q in qs],
        2.0 * T * (heads * (dq + dim) + ld), att + 4.0 * T * R * heads * dim)
    put(f"{tag}/expand_keys_values", [lambda: torch.mm(cache[0, :, :R], ukv.t())] * 5, 2.0 * T * (R + 2 * heads * dim), 4.0 * T * R * heads * dim)
    put(f"{tag}/rotate_queries", [lambda q=q: ops.rotate(q, q, heads, dim, dim, rot, trig, pos, T) for q in qs], 4.0 * T * heads * rot)
    z, qn, kn = rnd(T, qr + ld), f32(qr), f32(R)
    put(f"{tag}/latent_norms_append", [lambda: ops.latent_prep(z, 0, qn, pos, T, eps, cache, qr, kn, R, rot, trig)] * 5, 4.0 * T * (qr + ld))
    del qs
    ws, bias = [rnd(2 * ff, width, scale=width ** -0.5) for _ in range(3)], f32(2 * ff)
    nb, fl = 2.0 * (T * (width + ff) + 2 * ff * width), 4.0 * T * ff * width
    put(f"{tag}/dense_up_clamped", [lambda w=w: ops.gated_linear(h, w, bias, clamp) for w in ws], nb, fl)
    put(f"{tag}/dense_up_vendor_gemm_alone", [lambda w=w: ops.linear(h, w) for w in ws], nb + 2.0 * T * ff, fl)
    del ws
    put(f"{tag}/experts", [lambda i=i: ops.expert_rows(h, rw, rb, top, up[i], down[i], silu) for i in range(2)],
        2.0 * (3 * E * fe * width + T * width * (1 + top)), 6.0 * T * top * fe * width)
    rows, counts = rnd(T * top, width), torch.full((E,), T * top // E, dtype=torch.int32, device=dev)
    put(f"{tag}/expert_up_gemm", [lambda i=i: ops.group_gemm(rows, up[i], counts, gate=silu) for i in range(2)],
        2.0 * (2 * E * fe * width + T * top * (width + fe)), 4.0 * T * top * fe * width)
    act = rnd(T * top, fe)
    put(f"{tag}/expert_down_gemm", [lambda i=i: ops.group_gemm(act, down[i], counts) for i in range(2)],
        2.0 * (E * fe * width + T * top * (width + fe)), 2.0 * T * top * fe * width)
    return out


def run_sidirax_arm(args):
    import torch
    torch.cuda.set_device(0)
    sampler = ClockSampler(0)
    sampler.start()
    res = {}
    for size in KEPOVIK_SIZES:
        res[size] = {"layers": KEPOVIK_SIZES[size][-1], "kernels": sidirax_kernels(torch, size, args)}
        res[size]["kernels"]["kepovik"] = kepovik_kernels(torch, size, args)["kepovik"]
        if not args.headline_only:
            res[size].update(sidirax=model_speed(torch, sidirax_model, size, args), kepovik=model_speed(torch, kepovik_model, size, args))
    clocks = sampler.stop()
    best = res["2560"].get("sidirax", {}).get("prompt512_batch1", {})
    line = {"metric": "sidirax_decode_tokens_per_s", "value": best.get("decode_tokens_per_s"), "unit": "tokens/s", "n_gpus": 1,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": best.get("decode_ms"), "higher_is_better": True, "scaling": "weak",
            "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
            "config": {"workload": "sidirax_2560_30_layers_prompt512_batch1", "vocab": KEPOVIK_VOCAB, "experts": SIDIRAX_EXPERTS, "top": SIDIRAX_TOP,
                       "kv_rank": SIDIRAX_KV_RANK, "rot_dim": SIDIRAX_ROT, "decay_rank": KEPOVIK_RANK, "seed": args.seed,
                       "l2_policy": "weights, states and caches larger than L2 in rotation; decode activations stay in L2"},
            "sizes": res, "clocks": clocks}
    print(json.dumps(line), flush=True)


def _finish(world):
    """Leave without tearing NCCL down: destroying a process group while CUDA
    graphs that hold NCCL kernels are alive blocks at exit, so every rank meets
    at a barrier, flushes and exits the process directly."""
    if world > 1:
        import torch
        import torch.distributed as dist
        torch.cuda.synchronize()
        dist.barrier()
        torch.cuda.synchronize()
        sys.stdout.flush()
        sys.stderr.flush()
        os._exit(0)


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=100)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--tokens", type=int, default=8)
    ap.add_argument("--layers", type=int, default=30)
    ap.add_argument("--seed", type=int, default=1234)
    ap.add_argument("--workload", default="sweep", choices=["sweep", "tp", "decode", "list", "head", "prefill", "kepovik", "sidirax"])
    ap.add_argument("--unfused", action="store_true", help="decode workload: plain torch glue between the linears")
    ap.add_argument("--tp_mode", default="single", choices=["single", "fused", "exact"])
    ap.add_argument("--no_graph", action="store_true", help="tp workload: launch eagerly instead of replaying a CUDA graph")
    ap.add_argument("--verbose", action="store_true")
    ap.add_argument("--headline_only", action="store_true",
                    help="sweep workload: only the headline and end-to-end legs (short runs for profiling); sidirax workload: only the kernels")
    args = ap.parse_args()
    args.warmup = max(args.warmup, 3)
    if args.impl == "reference":
        run_reference_arm(args)
    elif args.workload == "tp":
        run_tp_arm(args)
    elif args.workload == "decode":
        run_decode_arm(args)
    elif args.workload == "kepovik":
        run_kepovik_arm(args)
    elif args.workload == "sidirax":
        run_sidirax_arm(args)
    elif args.workload in ("list", "head", "prefill"):
        run_single_leg(args)
    else:
        run_gpu_arm(args)


if __name__ == "__main__":
    main()
