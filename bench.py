"""Benchmark of the AWQ W4A16 linear path on B200.

Workload ("w4a16_gemm_sweep"): the 30-point GEMM shape sweep at group size 128,
M in {1, 4, 16, 128, 1024, 4096} x (K, N) in {(4096,4096), (4096,12288),
(12288,4096), (5120,25600), (25600,5120)}, fp16, seeded synthetic inputs with
the benchmark's distributions (int4 weights and zero-points uniform in [0,15],
scales uniform in [1e-3,1e-2], activations N(0,1)).  One step is one pass over
all 30 points; the metric is the time of that pass in microseconds (lower is
better).  Weights rotate over enough distinct copies per shape that a call
never finds its weights in L2.

  python bench.py [--gpus N] [--steps K] [--warmup W] [--impl reference]

With --gpus N > 1 (launched by torch.distributed.run) the same sweep runs
tensor-parallel: column-parallel shards along N, row-parallel shards along K on
group boundaries followed by an NCCL all-reduce (strong scaling).

--impl reference times the CPU restatement of the reference arithmetic (unpack
by shifts, (q - z) * s, fp32 matmul) on the host cores: every step is one real
pass over all 30 points.

On one GPU the line also carries `reference_gpu`: the reference's own
WQLinear_GEMM.forward (its Triton kernels, JIT-compiled on this GPU, and
torch.matmul) from the untracked install under baseline/_ref, on the same
tensors, after the timed regions.  With N > 1 it carries `tp_parity`: the
tensor-parallel results checked against the CPU oracle after the timed regions.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

import torch  # noqa: E402

MS = (1, 4, 16, 128, 1024, 4096)
# (K, N, how the layer is sharded under tensor parallelism)
SHAPES = ((4096, 4096, "column"), (4096, 12288, "column"), (12288, 4096, "row"),
          (5120, 25600, "column"), (25600, 5120, "row"))
GROUP = 128
L2_BYTES = 126 * 1024 * 1024


def weight_bytes(K, N, g=GROUP):
    return K * N // 2 + 2 * (K // g) * N + 4 * (K // g) * (N // 8)


def algo_bytes(M, K, N, g=GROUP):
    return weight_bytes(K, N, g) + 2 * M * K + 2 * M * N


def algo_flops(M, K, N):
    return 2 * M * N * K


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        p = json.load(open(path))
        return {"hbm_gbs": p["hbm_gbs"], "tflops_burst": p["bf16_tflops"],
                "tflops_sustained": p["bf16_tflops_sustained"], "source": "measured"}
    return {"hbm_gbs": 6650.0, "tflops_burst": 1590.0, "tflops_sustained": 1400.0, "source": "fallback"}


# --------------------------------------------------------------------------
# clocks sampled during the timed region
# --------------------------------------------------------------------------
class ClockSampler:
    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int):
        self.index, self.proc, self.lines = index, None, []

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", str(self.index), f"--query-gpu={self.Q}",
                                          "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
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
        except subprocess.TimeoutExpired:
            self.proc.kill()
        sm, mx, reasons = [], None, set()
        names = ("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap")
        for ln in self.lines:
            f = [x.strip() for x in ln.split(",")]
            if len(f) < 6:
                continue
            try:
                sm.append(float(f[0])); mx = float(f[1])
            except ValueError:
                continue
            for nm, v in zip(names, f[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(nm)
        sm.sort()
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": mx, "reasons": sorted(reasons),
                "samples": len(sm)}


# --------------------------------------------------------------------------
# our arm
# --------------------------------------------------------------------------
def shard_shape(K, N, kind, world):
    if world == 1:
        return K, N
    if kind == "column":
        return K, N // world
    return K // world, N


def make_layer(K, N, seed, dev, dtype):
    """A WQLinear_GEMM filled on the device with the benchmark's distributions."""
    import nanoquantization_b200 as nq
    lin = nq.WQLinear_GEMM(4, GROUP, K, N, dev, False, dtype)
    fill_layer(lin, seed, dev, dtype)
    return lin


def fill_layer(lin, seed, dev, dtype):
    g = torch.Generator(device=dev)
    g.manual_seed(seed)
    K, N = lin.in_features, lin.out_features
    # uniform 32-bit words = uniform nibbles, i.e. int4 weights / zero-points uniform in [0, 15]
    lin.qweight.copy_(torch.randint(-2 ** 31, 2 ** 31, (K, N // 8), generator=g, device=dev, dtype=torch.int64).to(torch.int32))
    lin.qzeros.copy_(torch.randint(-2 ** 31, 2 ** 31, (K // GROUP, N // 8), generator=g, device=dev, dtype=torch.int64).to(torch.int32))
    lin.qscales.copy_((torch.rand(K // GROUP, N, generator=g, device=dev) * 9e-3 + 1e-3).to(dtype))


def make_tp_layer(K, N, kind, world, rank, seed, dev, dtype):
    """The rank's shard of a (K, N) layer as the tensor-parallel class that an engine would use;
    the shard is filled directly (random init) instead of being sliced from a full tensor."""
    import nanoquantization_b200 as nq
    if kind == "column":
        lin = nq.ColumnParallelWQLinear(4, GROUP, K, N, world, rank, dev, False, dtype)
    else:
        lin = nq.RowParallelWQLinear(4, GROUP, K, N, world, rank, dev, False, dtype)
    fill_layer(lin.shard, seed, dev, dtype)
    return lin


def run_ours(args):
    import torch.distributed as dist
    import nanoquantization_b200 as nq  # noqa: F401
    from nanoquantization_b200 import _lib

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    if args.gpus != world:
        if world == 1 and args.gpus > 1:
            raise SystemExit("launch with torch.distributed.run for --gpus > 1")
    torch.cuda.set_device(local)
    dev = torch.device("cuda", local)
    stage = ["set-up"]
    if world > 1:
        if os.environ.get("NCCL_DEBUG", "VERSION").upper() == "VERSION":
            os.environ["NCCL_DEBUG"] = "WARN"  # keep NCCL's version banner out of stdout: one JSON line only
        # A rank may leave through a watchdog below while others are still inside a collective: keep NCCL off
        # NVLink multicast objects, which a vanished rank must not be bound to.
        os.environ.setdefault("NCCL_NVLS_ENABLE", "0")
        dist.init_process_group("nccl", device_id=dev)

        def give_up():
            # a multi-rank run that has not finished by now is stuck (one rank failed, the others wait for it)
            if rank == 0:
                emit(json.dumps({"metric": "w4a16_gemm_sweep_us", "n_gpus": world, "impl": "ours",
                                 "unavailable": f"the run did not finish within {args.max_seconds} s (stage: {stage[0]})"}))
            os._exit(0)
        overall = threading.Timer(args.max_seconds, give_up)
        overall.daemon = True
        overall.start()
    dtype = torch.float16
    lib = _lib.load()
    assert lib.nqb200_device_supported(local) == 1, "not a B200"

    # layers: enough copies per shape that one pass over the copies exceeds L2
    layers, xs_dev, xs_host, ys_host = {}, {}, {}, {}
    for si, (K, N, kind) in enumerate(SHAPES):
        k, n = shard_shape(K, N, kind, world)
        ncopy = max(2, -(-int(1.5 * L2_BYTES) // weight_bytes(k, n)))
        if world == 1:
            layers[si] = [make_layer(k, n, 1000 * si + c, dev, dtype) for c in range(ncopy)]
        else:
            layers[si] = [make_tp_layer(K, N, kind, world, rank, 1000 * si + c + 17 * rank, dev, dtype) for c in range(ncopy)]
        for M in MS:
            g = torch.Generator(device="cpu"); g.manual_seed(M * 31 + si)
            xh = torch.randn(M, k, generator=g).to(dtype).pin_memory()
            xs_host[(si, M)] = xh
            xs_dev[(si, M)] = xh.to(dev)
            ys_host[(si, M)] = torch.empty(M, n, dtype=dtype).pin_memory()
    points = [(si, M) for M in MS for si in range(len(SHAPES))]  # M-major: a shape's reuses are far apart

    # tensor parallelism: the row-parallel layers all-reduce over peer memory (inside the GEMM's finishing
    # kernel for decode sizes, stand-alone peer kernels above that, NCCL beyond the communicator's slot size)
    comm = None
    if world > 1 and not args.nccl_only:
        from nanoquantization_b200.layers.peer_comm import PeerAllReduce
        comm = PeerAllReduce(slot_bytes=2 << 20, num_slots=8, large_bytes=48 << 20, wait_limit_s=10.0)
        for si in layers:
            for lin in layers[si]:
                if hasattr(lin, "attach_comm"):
                    lin.attach_comm(comm)

    def call(si, M, copy, x):
        return layers[si][copy % len(layers[si])](x)  # row-parallel layers all-reduce inside

    # point j of a shape uses weight copy j, so a copy is reused only after the rest of the sweep
    # (>1 GB of other weights) has gone through L2
    def sweep_device(step=0):
        for j, (si, M) in enumerate(points):
            call(si, M, j // len(SHAPES) + step, xs_dev[(si, M)])

    # End to end: every point's activations come from pinned host memory and its result goes back to
    # pinned host memory inside the timed region, through WQLinear_GEMM.forward.  Three streams (copy in,
    # compute, copy out) so that a point's transfers overlap its neighbours' GEMMs, as a serving host would
    # drive a PCIe-attached GPU.
    s_in, s_mm, s_out = torch.cuda.Stream(), torch.cuda.Stream(), torch.cuda.Stream()
    ev_in = [torch.cuda.Event() for _ in points]
    ev_mm = [torch.cuda.Event() for _ in points]
    used = [False] * len(points)

    def sweep_e2e(step):
        for j, (si, M) in enumerate(points):
            with torch.cuda.stream(s_in):
                if used[j]:
                    s_in.wait_event(ev_mm[j])       # the previous step's GEMM still reads this buffer
                xs_dev[(si, M)].copy_(xs_host[(si, M)], non_blocking=True)
                ev_in[j].record(s_in)
            with torch.cuda.stream(s_mm):
                s_mm.wait_event(ev_in[j])
                y = call(si, M, j // len(SHAPES) + step, xs_dev[(si, M)])
                ev_mm[j].record(s_mm)
            used[j] = True
            with torch.cuda.stream(s_out):
                s_out.wait_event(ev_mm[j])
                y.record_stream(s_out)
                ys_host[(si, M)].copy_(y, non_blocking=True)

    def e2e_begin():
        cur = torch.cuda.current_stream()
        for st in (s_in, s_mm, s_out):
            st.wait_stream(cur)

    def e2e_end():
        cur = torch.cuda.current_stream()
        for st in (s_in, s_mm, s_out):
            cur.wait_stream(st)

    def barrier():
        torch.cuda.synchronize()
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    def capture(fn):
        """The launches of fn() as one CUDA graph (decode-sized calls are launch-bound from Python)."""
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            fn()
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            fn()
        return graph

    def timed(fn, steps, begin=None, end=None):
        barrier()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        if begin:
            begin()
        for s in range(steps):
            fn(s)
        if end:
            end()
        e1.record()
        barrier()
        ms = e0.elapsed_time(e1)
        if world > 1:
            t = torch.tensor([ms], device=dev)
            dist.all_reduce(t, op=dist.ReduceOp.MAX)
            ms = float(t.item())
        return ms

    use_graph = True
    try:
        sweep_graph = capture(sweep_device)  # with tensor parallelism the NCCL all-reduces are captured too
    except RuntimeError:
        if world == 1:
            raise
        use_graph, sweep_graph = False, None  # plain launches if this NCCL build refuses capture
        torch.cuda.synchronize()
    run_sweep = (lambda s: sweep_graph.replay()) if use_graph else sweep_device
    for w in range(max(args.warmup, 3)):
        run_sweep(w)
        e2e_begin(); sweep_e2e(w); e2e_end()
    sampler = ClockSampler(local)
    if rank == 0:
        sampler.start()
    stage[0] = "timed sweep"
    ms_dev = timed(run_sweep, args.steps)
    ms_e2e = timed(sweep_e2e, args.steps, e2e_begin, e2e_end)

    # per-point pass: each point launched back to back over rotating weight copies
    stage[0] = "per-point pass"
    per_point = []
    for (si, M) in points:
        K, N, kind = SHAPES[si]
        k, n = shard_shape(K, N, kind, world)
        reps = max(8, 2 * len(layers[si])) if M <= 128 else 4

        def burst(si=si, M=M, reps=reps):
            for r in range(reps):
                call(si, M, r, xs_dev[(si, M)])
        fn = capture(burst).replay if use_graph else burst
        for r in range(3):
            fn()
        barrier()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        us = e0.elapsed_time(e1) * 1e3 / reps
        per_point.append({"M": M, "K": k, "N": n, "us": us,
                          "kernel": lib.nqb200_gemm_kernel_name(M, n, k, GROUP, 0).decode()})
    clocks = sampler.stop() if rank == 0 else None
    barrier()
    # checker legs, after every timed region
    ref_gpu = tp_parity = None
    if world == 1 and not args.no_reference_gpu:
        ref_gpu = reference_gpu_leg(layers, xs_dev, points, per_point, dev)
    if world > 1:
        if comm is not None:
            for si in layers:
                for lin in layers[si]:
                    if hasattr(lin, "attach_comm"):
                        lin.attach_comm(None)
        stage[0] = "tp_parity"
        tp_parity = tp_parity_leg(world, rank, dev, dtype, comm)
        barrier()
    sweep_graph = fn = None  # graphs hold captured collectives: dropped well before the process group is destroyed
    decode, small, serve = None, None, None
    if not args.no_decode:
        for k in list(layers):
            del layers[k]
        torch.cuda.empty_cache()
        stage[0] = "decode_qwen3_8b"
        decode = decode_bench(world, rank, dev, dtype)
        barrier()
        if world == 1:
            torch.cuda.empty_cache()
            small = engine_bench_0p6b(dev, dtype)

    if rank == 0:
        pk = peaks()
        for p in per_point:
            gbs = algo_bytes(p["M"], p["K"], p["N"]) / p["us"] / 1e3
            tfl = algo_flops(p["M"], p["K"], p["N"]) / p["us"] / 1e6
            p.update({"gbs": round(gbs, 1), "tflops": round(tfl, 2), "hbm_frac": round(gbs / pk["hbm_gbs"], 4),
                      "tensor_frac": round(tfl / pk["tflops_burst"], 4), "us": round(p["us"], 2)})

        def agg(sel, kind):
            pts = [p for p in per_point if sel(p)]
            t = sum(p["us"] for p in pts)
            if kind == "hbm":
                a = sum(algo_bytes(p["M"], p["K"], p["N"]) for p in pts) / t / 1e3
                return {"bound": "hbm", "achieved": round(a, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                        "frac": round(a / pk["hbm_gbs"], 4), "traffic": None, "peak_source": pk["source"],
                        "kernel": pts[0]["kernel"], "points": len(pts)}
            a = sum(algo_flops(p["M"], p["K"], p["N"]) for p in pts) / t / 1e6
            return {"bound": "tensor", "achieved": round(a, 1), "peak": pk["tflops_burst"], "unit": "TFLOP/s",
                    "frac": round(a / pk["tflops_burst"], 4), "traffic": None, "peak_source": pk["source"],
                    "kernel": pts[0]["kernel"], "points": len(pts)}

        # the kernel where the sweep's time goes (about 90 % of the launch-list time): the tcgen05 prefill
        # kernel on its tensor-bound points (M >= 1024)
        dom = per_point[-1]["kernel"]
        roof_prefill = agg(lambda p: p["kernel"] == dom and p["M"] >= 1024, "tensor")
        dom_pts = [p for p in per_point if p["kernel"] == dom and p["M"] >= 1024]
        # DRAM bytes per launch, from the ncu capture of this kernel at M = K = N = 4096 (profiles/): reads 1.19 x
        # the algorithmic read bytes (packed weights + activations), writes 0.32 x the output (the rest is still
        # in L2 when the kernel ends); scaled to the points of the sweep in proportion to those bytes
        roof_prefill["traffic"] = round(sum(1.19 * (weight_bytes(p["K"], p["N"]) + 2 * p["M"] * p["K"]) + 0.32 * 2 * p["M"] * p["N"]
                                            for p in dom_pts) / len(dom_pts))
        roof_prefill["traffic_unit"] = "bytes per launch (mean over the kernel's points)"
        roof_decode = agg(lambda p: p["M"] <= 16, "hbm")
        # ncu: both decode kernels read exactly their algorithmic bytes from DRAM (profiles/)
        roof_decode["traffic"] = round(sum(algo_bytes(p["M"], p["K"], p["N"]) for p in per_point if p["M"] <= 16) / 15)
        h2d = sum(2 * M * shard_shape(*SHAPES[si], world)[0] for (si, M) in points)
        d2h = sum(2 * M * shard_shape(*SHAPES[si], world)[1] for (si, M) in points)
        us_step = ms_dev * 1e3 / args.steps
        line = {
            "metric": "w4a16_gemm_sweep_us", "value": round(us_step, 2), "unit": "us", "n_gpus": world,
            "steps": args.steps, "warmup": max(args.warmup, 3), "ms_per_step": round(us_step / 1e3, 4),
            "higher_is_better": False, "scaling": "strong", "vs_baseline": None,
            "dtype": "f16", "data": "synthetic",
            "config": sweep_config(f"tp{world}",
                                   ("device-timed sweep replayed as one CUDA graph" if use_graph else "plain launches") +
                                   "; e2e through WQLinear_GEMM.forward, host<->device copies on their own streams"),
            "e2e": {"value": round(ms_e2e * 1e3 / args.steps, 2), "unit": "us", "h2d_bytes_per_step": h2d,
                    "d2h_bytes_per_step": d2h},
            "gpu_launches": args.steps * sum(lib.nqb200_gemm_launch_count(M, *shard_shape(*SHAPES[si], world)[::-1], GROUP, 0)
                                             for (si, M) in points),
            "roofline": roof_prefill, "roofline_decode": roof_decode,
            "clocks": clocks, "points": per_point, "decode_qwen3_8b": decode, "engine_qwen3_0p6b": small,
        }
        if ref_gpu is not None:
            line["reference_gpu"] = ref_gpu
        if tp_parity is not None:
            line["tp_parity"] = tp_parity
        if world == 1:
            line["cpu_baseline"] = cpu_baseline()
    if world == 8 and not args.no_serve and not args.no_decode:
        # The largest configuration: Qwen3-32B architecture, 256 requests, continuous batching, on all 8 GPUs.  The
        # line above stands whatever happens here: past its time budget every rank leaves, rank 0 printing the line
        # without this part (ranks that wait in a collective for one that failed would wait for NCCL's own
        # time-out, ten minutes).
        stage[0] = "serve"
        lock, printed = threading.Lock(), [False]

        def serve_over_budget():
            with lock:
                if printed[0]:
                    return
                printed[0] = True
                if rank == 0:
                    line["serve_qwen3_32b"] = {"unavailable": f"did not finish within {args.serve_budget} s"}
                    emit(json.dumps(line))
            os._exit(0)
        timer = threading.Timer(args.serve_budget, serve_over_budget)
        timer.daemon = True
        timer.start()
        torch.cuda.empty_cache()
        try:
            serve = serve_bench(world, rank, dev, dtype)
        except Exception as exc:
            serve = {"error": f"{type(exc).__name__}: {exc}"[:300]}
        barrier()
        with lock:
            printed[0] = True
        timer.cancel()
        if rank == 0:
            line["serve_qwen3_32b"] = serve
    if rank == 0:
        emit(json.dumps(line))
    stage[0] = "teardown"
    if comm is not None:
        comm.close()
    leave_distributed(world)
    if world > 1:
        overall.cancel()


def sweep_config(parallelism, launch):
    """The `config` object, the same keys in both arms."""
    return {"workload": "w4a16_gemm_sweep g128 M{1,4,16,128,1024,4096} x 5 (K,N) shapes (config 2)",
            "points_per_step": len(MS) * len(SHAPES), "parallelism": parallelism,
            "l2": "weights rotate over copies totalling >1.5x L2 per shape", "launch": launch}


def leave_distributed(world):
    """Tear the process group down.  Captured CUDA graphs hold NCCL kernels of the communicator, so every
    graph is dropped (and collected) and the device is idle before the communicator is destroyed; a
    watchdog ends the process if the teardown still does not return."""
    if world <= 1:
        return
    import gc
    import torch.distributed as dist
    torch.cuda.synchronize()
    dist.barrier()
    gc.collect()
    torch.cuda.synchronize()
    sys.stdout.flush()
    sys.stderr.flush()
    watchdog = threading.Timer(30.0, lambda: os._exit(0))
    watchdog.daemon = True
    watchdog.start()
    dist.destroy_process_group()
    watchdog.cancel()


# --------------------------------------------------------------------------
# second half of the metric: Qwen3-8B-architecture AWQ decode tokens/s through the engine
# --------------------------------------------------------------------------
def engine_bench_0p6b(dev, dtype, prompts=32, prompt_len=512, steps=256):
    """Random-init Qwen3-0.6B (w4 g128) on one GPU through LLMEngine.generate: 32 prompts of 512 random
    ids, 256 greedy tokens each (prefill, then decode steps as CUDA graphs)."""
    from nanoquantization_b200 import WQLinear_GEMM
    from nanoquantization_b200.engine import LLMEngine
    from nanoquantization_b200.models import QWEN3_SHAPES, Qwen3QuantizedForCausalLM
    shp = QWEN3_SHAPES["qwen3-0.6b"]
    model = Qwen3QuantizedForCausalLM(shp["num_hidden_layers"], 151936, shp["hidden_size"], shp["total_num_heads"],
                                      shp["total_num_kv_heads"], 8192, shp["intermediate_size"], 4, GROUP, 128, False, 1e6,
                                      1e-6, device=dev, dtype=dtype)
    n = 0
    for mod in model.modules():
        if isinstance(mod, WQLinear_GEMM):
            fill_layer(mod, 9000 + n, dev, dtype)
            n += 1
    torch.nn.init.normal_(model.model.embed_tokens.weight, std=0.02)
    torch.nn.init.normal_(model.lm_head.weight, std=0.02)
    model.fuse_projections()
    block = 256
    per_seq = -(-(prompt_len + steps + 8) // block)
    eng = LLMEngine(model, num_blocks=prompts * per_seq + 4, block_size=block, max_batch=prompts)
    g = torch.Generator().manual_seed(2)
    ids = [torch.randint(0, 151936, (prompt_len,), generator=g).tolist() for _ in range(prompts)]
    eng.generate(ids[:prompts], 4)  # warm-up: graphs captured, workspaces allocated
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    outs = eng.generate(ids, steps)
    torch.cuda.synchronize()
    dt = time.perf_counter() - t0
    new = sum(len(o) for o in outs)
    return {"model": "qwen3-0.6b-arch w4 g128 random init", "prompts": prompts, "prompt_len": prompt_len,
            "new_tokens": new, "wall_s": round(dt, 3), "generated_tok_per_s": round(new / dt, 1),
            "total_tok_per_s": round((new + prompts * prompt_len) / dt, 1)}


def serve_bench(world, rank, dev, dtype, requests=256, arch="qwen3-32b", max_batch=64):
    """Continuous batching through LLMEngine.generate: random-init model of `arch` (w4 g128, tensor-parallel
    over `world` ranks), `requests` requests with prompt lengths uniform in [128, 4096] and output lengths
    uniform in [64, 512], random ids, greedy decoding: the benchmark's largest configuration, which names the
    32B architecture on 8 GPUs.  Part of the `--gpus 8` line; on its own as `bench.py --serve`."""
    import torch.distributed as dist
    from nanoquantization_b200 import WQLinear_GEMM
    from nanoquantization_b200.engine import LLMEngine
    from nanoquantization_b200.models import QWEN3_SHAPES, Qwen3QuantizedForCausalLM
    shp = QWEN3_SHAPES[arch]
    model = Qwen3QuantizedForCausalLM(shp["num_hidden_layers"], 151936, shp["hidden_size"], shp["total_num_heads"],
                                      shp["total_num_kv_heads"], 8192, shp["intermediate_size"], 4, GROUP, 128, False, 1e6,
                                      1e-6, tp_size=world, tp_rank=rank, device=dev, dtype=dtype)
    n = 0
    for mod in model.modules():
        if isinstance(mod, WQLinear_GEMM):
            fill_layer(mod, 7000 + n + 100 * rank, dev, dtype)
            n += 1
    torch.nn.init.normal_(model.model.embed_tokens.weight, std=0.02)
    torch.nn.init.normal_(model.lm_head.weight, std=0.02)
    model.fuse_projections()
    comm = None
    if world > 1:
        from nanoquantization_b200.layers.peer_comm import PeerAllReduce
        comm = PeerAllReduce(slot_bytes=2 << 20, num_slots=8, large_bytes=48 << 20, wait_limit_s=10.0)
        model.attach_peer_comm(comm)
    g = torch.Generator().manual_seed(11)   # the same requests on every rank
    plen = torch.randint(128, 4097, (requests,), generator=g).tolist()
    olen = torch.randint(64, 513, (requests,), generator=g).tolist()
    prompts = [torch.randint(0, 151936, (n_,), generator=g).tolist() for n_ in plen]
    block = 256
    eng = LLMEngine(model, num_blocks=max_batch * (-(-(4096 + 512 + 8) // block)) + 4, block_size=block, max_batch=max_batch,
                    max_prefill_tokens=8192)
    eng.generate([p[:300] for p in prompts[:max_batch]], 3)   # warm-up: workspaces, first graphs
    torch.cuda.synchronize()
    if world > 1:
        dist.barrier()
    t0 = time.perf_counter()
    outs = eng.generate(prompts, olen)
    torch.cuda.synchronize()
    dt = time.perf_counter() - t0
    if world > 1:
        t = torch.tensor([dt], device=dev, dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        dt = float(t.item())
    new = sum(len(o) for o in outs)
    assert [len(o) for o in outs] == olen
    out = {"workload": f"{arch}-arch w4 g128 random init, continuous batching", "tp": world, "requests": requests,
           "prompt_tokens": sum(plen), "new_tokens": new, "max_batch": max_batch, "wall_s": round(dt, 2),
           "generated_tok_per_s": round(new / dt, 1), "total_tok_per_s": round((new + sum(plen)) / dt, 1),
           "decode_graphs": len(eng._graphs)}
    if comm is not None:
        out["peer_allreduce_status"] = comm.status()
    return out


def decode_bench(world, rank, dev, dtype, batches=(1, 16, 64), context=2048, steps=16, prefill=True):
    """Random-init Qwen3-8B (w4 g128, tensor-parallel over `world` ranks), sequences with a
    2048-token context in the paged KV cache, greedy decode steps replayed as a CUDA graph."""
    import torch.distributed as dist
    from nanoquantization_b200 import WQLinear_GEMM
    from nanoquantization_b200.engine import LLMEngine, Sequence
    from nanoquantization_b200.models import QWEN3_SHAPES, Qwen3QuantizedForCausalLM
    shp = QWEN3_SHAPES["qwen3-8b"]
    model = Qwen3QuantizedForCausalLM(shp["num_hidden_layers"], 151936, shp["hidden_size"], shp["total_num_heads"],
                                      shp["total_num_kv_heads"], 8192, shp["intermediate_size"], 4, GROUP, 128, False, 1e6,
                                      1e-6, tp_size=world, tp_rank=rank, device=dev, dtype=dtype)
    n = 0
    for mod in model.modules():
        if isinstance(mod, WQLinear_GEMM):
            fill_layer(mod, 5000 + n + 100 * rank, dev, dtype)
            n += 1
    torch.nn.init.normal_(model.model.embed_tokens.weight, std=0.02)
    torch.nn.init.normal_(model.lm_head.weight, std=0.02)
    model.fuse_projections()
    block = 256
    per_seq = -(-(context + steps + 8) // block)
    eng = LLMEngine(model, num_blocks=max(batches) * per_seq + 4, block_size=block, max_batch=max(batches))
    out = {"model": "qwen3-8b-arch w4 g128 random init", "tp": world, "context": context,
           "allreduce_variants": "nccl = NCCL after each row-parallel linear; peer = nqb200_gemm_allreduce "
                                 "(reduced over peer memory by the kernel that finishes the GEMM)",
           "attention": "flash_attn paged" if eng.paged_attention is not None else "sdpa over gathered pages", "points": []}
    g = torch.Generator().manual_seed(1)
    comm = None
    if world > 1:
        from nanoquantization_b200.layers.peer_comm import PeerAllReduce
        comm = PeerAllReduce(slot_bytes=1 << 20, num_slots=8, large_bytes=48 << 20, wait_limit_s=10.0)   # 72 all-reduces per step: a multiple of the slot count
    variants = [("nccl", None)] + ([("peer", comm)] if comm is not None else [])
    for (ar_name, ar_comm), B in [(v, b) for v in variants for b in batches]:
        model.attach_peer_comm(ar_comm)
        eng._graphs.clear()
        seqs = []
        for i in range(B):
            s = Sequence(i, torch.randint(0, 151936, (context,), generator=g).tolist(), 10 ** 9)
            assert eng.blocks.ensure(s, context + steps + 8)
            s.output.append(1)
            seqs.append(s)
        for _ in range(3):
            eng._decode(seqs)
        torch.cuda.synchronize()
        if world > 1:
            dist.barrier()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(steps):
            eng._decode(seqs)
        e1.record()
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1) / steps
        if world > 1:
            t = torch.tensor([ms], device=dev)
            dist.all_reduce(t, op=dist.ReduceOp.MAX)
            ms = float(t.item())
        pt = {"batch": B, "ms_per_step": round(ms, 3), "tok_per_s": round(B / ms * 1e3, 1)}
        if world > 1:
            pt["allreduce"] = ar_name
        if world > 1 and ar_name == "nccl":  # share of the step spent in the 2 all-reduces per layer
            buf = torch.zeros(B, shp["hidden_size"], dtype=dtype, device=dev)
            gr = torch.cuda.CUDAGraph()
            for _ in range(2 * shp["num_hidden_layers"]):
                dist.all_reduce(buf)
            torch.cuda.synchronize()
            with torch.cuda.graph(gr):
                for _ in range(2 * shp["num_hidden_layers"]):
                    dist.all_reduce(buf)
            gr.replay(); torch.cuda.synchronize()
            e0.record(); gr.replay(); e1.record(); torch.cuda.synchronize()
            pt["allreduce_ms_per_step"] = round(e0.elapsed_time(e1), 3)
            pt["allreduce_share"] = round(e0.elapsed_time(e1) / ms, 3)
        out["points"].append(pt)
        for s in seqs:
            eng.blocks.release(s)
    # the configuration's 4096-token prefill: one sequence through the engine's prefill path
    seq = Sequence(10 ** 6, torch.randint(0, 151936, (4096,), generator=g).tolist(), 1)
    if prefill and eng.blocks.ensure(seq, 4096 + 8):
        model.attach_peer_comm(None)
        for _ in range(2):
            eng._prefill([seq])
        torch.cuda.synchronize()
        if world > 1:
            dist.barrier()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(3):
            eng._prefill([seq])
        e1.record()
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1) / 3
        if world > 1:
            t = torch.tensor([ms], device=dev)
            dist.all_reduce(t, op=dist.ReduceOp.MAX)
            ms = float(t.item())
        out["prefill_4096"] = {"ms": round(ms, 3), "tok_per_s": round(4096 / ms * 1e3, 1)}
        eng.blocks.release(seq)
    if comm is not None:
        out["peer_allreduce_status"] = comm.status()
    del eng, model
    torch.cuda.empty_cache()
    return out


# --------------------------------------------------------------------------
# Vemedra: layers of a real model's size beside the Qwen3 layers of the same size (--vemedra)
# --------------------------------------------------------------------------
VEMEDRA_LAYERS = 8


def vemedra_config(layers=VEMEDRA_LAYERS, chunk=4096):
    """Widths of the Qwen3-8B architecture: 4096 wide, 32 query heads over 8, head size 128, feed-forward 12288; every
    fourth layer a minGRU, the others attention in chunks beside 16 retention heads."""
    ff = {"kind": "dense", "ff": 12288, "limit": 7.0}
    gru = {"type": "mingru", "mixer": {"width": 4096}, "mlp": ff}
    par = {"type": "parallel", "mlp": ff, "mixer": {
        "left": {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "mask": {"size": chunk}, "rot": {"base": 1e6, "dims": 128},
                 "scale": 128 ** -0.5, "softcap": 50.0},
        "right": {"heads": 16, "dim": 128, "vdim": 256, "decay": [1 - 2.0 ** -(5 + 0.5 * h) for h in range(16)]}, "left_scale": 1.0, "right_scale": 0.5}}
    return {"architecture": "Vemedra", "vocab": 151936, "width": 4096, "canon": {"taps": 4}, "norm": {"eps": 1e-6},
            "layers": [gru if i % 4 == 0 else par for i in range(layers)]}


def _device_us(fn, reps):
    """Microseconds per call of ``fn(i)``, i = 0 .. reps - 1, replayed as one CUDA graph."""
    fn(0)
    torch.cuda.synchronize()
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        for i in range(reps):
            fn(i)
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for i in range(reps):
            fn(i)
    for _ in range(3):
        graph.replay()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(3):
        graph.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) * 1e3 / (3 * reps)


def _engine_throughput(eng, vocab, batches, context, prefill, steps=16):
    """Decode steps per batch size over a given context, and one prompt, as in the Qwen3-8B section."""
    from nanoquantization_b200.engine import Sequence
    g = torch.Generator().manual_seed(1)
    out = {"decode": [], "context": context}
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    for B in batches:
        eng._graphs.clear()
        seqs = []
        for i in range(B):
            s = Sequence(i, torch.randint(0, vocab, (context,), generator=g).tolist(), 10 ** 9)
            eng._hold(s, context + 8)
            s.output.append(s.prompt[0])      # unlike tokens: a router sends them to unlike experts
            seqs.append(s)
        for _ in range(3):
            eng._decode(seqs)
        torch.cuda.synchronize()
        e0.record()
        for _ in range(steps):
            eng._decode(seqs)
        e1.record()
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1) / steps
        graph = next(iter(eng._graphs.values()))[0]
        e0.record()
        for _ in range(steps):
            graph.replay()
        e1.record()
        torch.cuda.synchronize()
        out["decode"].append({"batch": B, "ms_per_step": round(ms, 3), "tok_per_s": round(B / ms * 1e3, 1),
                              "graph_ms": round(e0.elapsed_time(e1) / steps, 3)})
        for s in seqs:
            eng.drop(s)
    eng._graphs.clear()
    seq = Sequence(10 ** 6, torch.randint(0, vocab, (prefill,), generator=g).tolist(), 1)
    times = []
    for k in range(5):
        eng._hold(seq, prefill + 1)
        torch.cuda.synchronize()
        e0.record()
        eng._prefill([seq])
        e1.record()
        torch.cuda.synchronize()
        times.append(e0.elapsed_time(e1))
        eng.drop(seq)
    ms = sorted(times[2:])[1]
    out["prefill"] = {"tokens": prefill, "ms": round(ms, 3), "tok_per_s": round(prefill / ms * 1e3, 1)}
    return out


def vemedra_kernels(dev, peaks, T=8192, context=2048):
    """Each kernel of a layer on its own, on inputs larger than L2 (rotating copies), against its roofline, and the
    kernels of a Qwen3 layer that do the like."""
    import torch.nn.functional as F
    from nanoquantization_b200.engine import StepBatch
    from nanoquantization_b200.layers import fused, mixers as ops
    from nanoquantization_b200.layers.sequence_mixers import AttentionMixer
    from nanoquantization_b200 import _lib
    hbm, bf16 = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    W, H, G, D, RH, RD, RV, FF, chunk, bs = 4096, 32, 8, 128, 16, 128, 256, 12288, 4096, 256
    rows = []
    dt = torch.bfloat16

    def rnd(*shape, dtype=dt):
        return torch.randn(*shape, device=dev, dtype=torch.float32).to(dtype)

    def add(phase, name, us, nbytes=0, flops=0):
        tb, tf = nbytes / hbm * 1e6, flops / bf16 * 1e6
        rows.append({"phase": phase, "kernel": name, "us": round(us, 2), "bound": "hbm" if tb >= tf else "tensor",
                     "of_roofline": round(max(tb, tf) / us, 3)})

    def step(n, B, start):
        blocks = -(-(start + n) // bs)
        return StepBatch.host([[0] * n] * B, [start] * B, [[b * blocks + i for i in range(blocks)] for b in range(B)], list(range(B)), blocks, bs).to(dev)
    one = step(T, 1, 0)
    nin = H * D + 2 * G * D + 2 * RH * RD + 2 * RH * RV
    att = AttentionMixer(heads=H, kv_heads=G, dim=D, vdim=D, chunk=chunk, rot_base=1e6, rot_dims=D, scale=D ** -0.5, softcap=50.0, device=dev)
    decay = torch.tensor([1 - 2.0 ** -(5 + 0.5 * h) for h in range(RH)], device=dev)
    ret = _lib.RetentionDesc(RH, RD, RV, 1e-6, 0.5, decay.data_ptr())
    # prefill
    x, nw, cw = [rnd(T, W, dtype=torch.float32) for _ in range(2)], rnd(W, dtype=torch.float32), rnd(4, W, dtype=torch.float32)
    cst = torch.zeros(65, 3, W, device=dev)
    add("prefill", "rmsnorm + convolution", _device_us(lambda i: ops.rmsnorm_conv(x[i % 2], nw, cw, cst, one, 1e-6, dt), 8), T * W * 6)
    x16, r16, n16 = [rnd(T, W) for _ in range(2)], [rnd(T, W) for _ in range(2)], rnd(W)
    add("prefill", "Qwen3: residual add + rmsnorm", _device_us(lambda i: fused.add_rmsnorm(x16[i % 2], r16[i % 2], n16, 1e-6), 8), T * W * 8)
    del r16
    proj = [rnd(T, nin) for _ in range(2)]
    kc, vc = torch.zeros(T // bs + 1, bs, G, D, dtype=dt, device=dev), torch.zeros(T // bs + 1, bs, G, D, dtype=dt, device=dev)
    add("prefill", "rotary + K/V store", _device_us(lambda i: ops.rope_store(proj[i % 2], kc, vc, att.inv_freq, one, 0, H * D, (H + G) * D, H), 8),
        T * (2 * H * D + 4 * G * D) * 2)
    qkv, qn, cs = [rnd(T, (H + 2 * G) * D) for _ in range(3)], rnd(D), rnd(T, 1, D, dtype=torch.float32)
    kq, vq = torch.zeros_like(kc), torch.zeros_like(vc)
    add("prefill", "Qwen3: QK-norm + rotary + K/V store",
        _device_us(lambda i: fused.qknorm_rope_(qkv[i % 3], qn, qn, cs, one.positions, H, G, D, 1e-6, (kq, vq, one.rows)), 9), T * (2 * H * D + 4 * G * D) * 2)
    act = rnd(T, H * D + RH * RV)
    for name, c, cap in ((f"attention, chunks of {chunk}", chunk, 50.0), ("attention, one chunk of all", T, 50.0), ("attention, the same with scores beyond the cap", T, 3.0)):
        att.chunk, att.softcap = c, cap
        d = att.desc()
        us = _device_us(lambda i: ops.chunk_attention(proj[i % 2][:, :H * D], kc, vc, act[:, :H * D], d, one), 4)
        add("prefill", name, us, flops=T // c * (c * c / 2) * 4 * D * H)
    att.softcap = 50.0
    q, k, v = (qkv[0][:, o:o + n * D].reshape(1, T, n, D).transpose(1, 2).contiguous() for o, n in ((0, H), (H * D, G), ((H + G) * D, G)))
    us = _device_us(lambda i: F.scaled_dot_product_attention(q, k, v, is_causal=True, enable_gqa=True), 4)
    add("prefill", "Qwen3: scaled_dot_product_attention, all", us, flops=T * T / 2 * 4 * D * H)
    del q, k, v, qkv
    st, off = torch.zeros(65, RH, RD, RV, device=dev), (H + 2 * G) * D
    us = _device_us(lambda i: ops.retention_gated(proj[i % 2], off, ret, decay, st, act, H * D, one), 4)
    add("prefill", "retention + norm + gate (3 launches)", us, T * (2 * RH * RD + 3 * RH * RV) * 2, 4 * T * RH * RD * RV)
    zb, gst, p3 = rnd(W, dtype=torch.float32), torch.zeros(65, W, device=dev), [rnd(T, 3 * W) for _ in range(2)]
    add("prefill", "minGRU scan", _device_us(lambda i: ops.mingru(p3[i % 2], W, zb, zb, gst, one), 8), T * W * 8)
    del p3
    gu = [rnd(T, 2 * FF) for _ in range(2)]
    add("prefill", "clamped GLU", _device_us(lambda i: ops.clamped_glu(gu[i % 2], 7.0), 8), T * FF * 6)
    add("prefill", "Qwen3: silu(gate) * up", _device_us(lambda i: fused.silu_mul(gu[i % 2]), 8), T * FF * 6)
    del gu
    w = rnd(nin, W)
    add("prefill", "merged input product (library)", _device_us(lambda i: ops.linear(x16[i % 2], w), 4), flops=2 * T * W * nin)
    w2 = rnd(W, FF)
    y = rnd(T, FF)
    add("prefill", "down product + residual (library)", _device_us(lambda i: ops.linear_residual_(x[i % 2], y, w2), 4), flops=2 * T * W * FF)
    lin = make_layer(W, 2 * FF, 11, dev, dt)
    add("prefill", "Qwen3: gate | up product, 4-bit weights", _device_us(lambda i: lin(x16[i % 2]), 4), flops=2 * T * W * 2 * FF)
    del proj, act, x, x16, y, w, w2, lin
    torch.cuda.empty_cache()
    # decode: the weights rotate over copies larger than L2
    for B in (1, 16):
        ph, h = f"decode, batch {B}", rnd(B, W)
        s = step(1, B, context - 1)
        stream, f12 = rnd(B, W, dtype=torch.float32), rnd(B, FF)
        ws = [rnd(nin, W) for _ in range(3)]
        add(ph, "merged input product", _device_us(lambda i: ops.linear(h, ws[i % 3]), 12), nin * W * 2)
        ws = [rnd(2 * FF, W) for _ in range(2)]
        add(ph, "gate | up product + clamped GLU", _device_us(lambda i: ops.dense_glu(h, ws[i % 2], 7.0), 8), 2 * FF * W * 2)
        ws = [rnd(W, FF) for _ in range(3)]
        add(ph, "down product + residual", _device_us(lambda i: ops.linear_residual_(stream, f12, ws[i % 3]), 12), FF * W * 2)
        ws = [rnd(W, H * D + RH * RV) for _ in range(4)]
        a8 = rnd(B, H * D + RH * RV)
        add(ph, "output product + residual", _device_us(lambda i: ops.linear_residual_(stream, a8, ws[i % 4]), 12), W * (H * D + RH * RV) * 2)
        ws = [rnd(3 * W, W) for _ in range(3)]
        add(ph, "z | x | g product + minGRU", _device_us(lambda i: ops.dense_mingru(h, ws[i % 3], zb, zb, gst, s), 12), 3 * W * W * 2)
        del ws
        for (K, N) in ((W, 2 * FF), (FF, W), (W, (H + 2 * G) * D)):
            n = max(2, -(-int(1.5 * L2_BYTES) // weight_bytes(K, N)))
            lins = [make_layer(K, N, 7 + c, dev, dt) for c in range(n)]
            xk = rnd(B, K)
            add(ph, f"Qwen3: 4-bit linear {K} -> {N}", _device_us(lambda i: lins[i % n](xk), 2 * n), weight_bytes(K, N))
            del lins
        n = 8 if B == 1 else 2   # copies of cache and state
        copies = []
        for _ in range(n):
            nb = B * (context // bs)
            copies.append((rnd(nb, bs, G, D), rnd(nb, bs, G, D), torch.zeros(B, RH, RD, RV, device=dev)))
        pr, ac = rnd(B, nin), rnd(B, H * D + RH * RV)
        att.chunk = chunk
        d = att.desc()
        kv_bytes, st_bytes = B * context * 2 * G * D * 2, 2 * B * RH * RD * RV * 4
        both = lambda i: ops.mixer_decode(pr, ac, (d, att.rope_desc(), 0, att.value_column(0), 0, copies[i % n][0], copies[i % n][1]), (ret, off, H * D, copies[i % n][2]), s)  # noqa: E731
        add(ph, "attention + retention", _device_us(both, 2 * n), kv_bytes + st_bytes)
        add(ph, "  attention alone", _device_us(lambda i: ops.mixer_decode(pr, ac, (d, att.rope_desc(), 0, att.value_column(0), 0, copies[i % n][0], copies[i % n][1]), None, s), 2 * n), kv_bytes)
        add(ph, "  retention alone", _device_us(lambda i: ops.mixer_decode(pr, ac, None, (ret, off, H * D, copies[i % n][2]), s), 2 * n), st_bytes)
        try:
            from flash_attn import flash_attn_with_kvcache
            q1 = rnd(B, 1, H, D)
            add(ph, "Qwen3: flash_attn_with_kvcache", _device_us(lambda i: flash_attn_with_kvcache(
                q1, copies[i % n][0], copies[i % n][1], cache_seqlens=s.ctx, block_table=s.table, causal=True), 2 * n), kv_bytes)
        except ImportError:
            pass
        add(ph, "rmsnorm + convolution", _device_us(lambda i: ops.rmsnorm_conv(stream, nw, cw, cst, s, 1e-6, dt), 16), B * W * (6 + 24) + W * 20)
        add(ph, "Qwen3: residual add + rmsnorm", _device_us(lambda i: fused.add_rmsnorm(h, h, n16, 1e-6), 16), B * W * 8)
        del copies
    return rows


def run_vemedra(args):
    """--vemedra: random-init layers of real sizes through the engine, beside Qwen3 layers (4-bit weights) of the same
    width, heads and feed-forward, and every kernel against its roofline."""
    from nanoquantization_b200 import WQLinear_GEMM
    from nanoquantization_b200.engine import LLMEngine
    from nanoquantization_b200.models import QWEN3_SHAPES, Qwen3QuantizedForCausalLM, VemedraConfig, VemedraForCausalLM
    torch.cuda.set_device(0)
    dev, dt = torch.device("cuda", 0), torch.bfloat16
    torch.manual_seed(0)
    with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as fh:
        peaks = json.load(fh)
    line = {"what": "Vemedra beside Qwen3 (4-bit weights), random init, one GPU, bf16", "layers": VEMEDRA_LAYERS,
            "note": "weights and caches larger than L2; rooflines are the measured copy bandwidth and bf16 peak"}
    sampler = ClockSampler(0)
    sampler.start()
    if not args.vemedra_kernels_only:
        batches, context, prefill = (1, 16, 64), 2047, 8192
        model = VemedraForCausalLM(VemedraConfig.from_dict(vemedra_config()), device=dev, dtype=dt)
        for name, t in model.checkpoint_tensors().items():
            if "norm" in name:
                t.fill_(1.0)
            else:
                t.copy_(torch.randn(t.shape, device=dev) * (t.shape[-1] ** -0.5 if t.dim() > 1 else 0.1))
        eng = LLMEngine(model, num_blocks=64 * 9 + 40, max_batch=64)
        line["vemedra"] = _engine_throughput(eng, 151936, batches, context, prefill)
        line["vemedra"]["weights_gb"] = round(sum(t.numel() * t.element_size() for t in model.buffers()) / 1e9, 2)
        del eng, model
        torch.cuda.empty_cache()
        shp = QWEN3_SHAPES["qwen3-8b"]
        model = Qwen3QuantizedForCausalLM(VEMEDRA_LAYERS, 151936, shp["hidden_size"], shp["total_num_heads"], shp["total_num_kv_heads"], 8400,
                                          shp["intermediate_size"], 4, GROUP, 128, False, 1e6, 1e-6, device=dev, dtype=dt)
        for n, mod in enumerate(m for m in model.modules() if isinstance(m, WQLinear_GEMM)):
            fill_layer(mod, 5000 + n, dev, dt)
        torch.nn.init.normal_(model.model.embed_tokens.weight, std=0.02)
        torch.nn.init.normal_(model.lm_head.weight, std=0.02)
        model.fuse_projections()
        eng = LLMEngine(model, num_blocks=64 * 9 + 40, max_batch=64)
        line["qwen3"] = _engine_throughput(eng, 151936, batches, context, prefill)
        del eng, model
        torch.cuda.empty_cache()
    line["kernels"] = vemedra_kernels(dev, peaks)
    line["clocks"] = sampler.stop()
    emit(json.dumps(line))


# --------------------------------------------------------------------------
# Verozen: layers of a real model's size beside the Vemedra layers of the same size (--verozen)
# --------------------------------------------------------------------------
VEROZEN_LAYERS = 8
VEROZEN_EXPERTS = {"experts": 64, "top": 8, "groups": {"count": 8, "keep": 4}, "scale": 2.5}
VEROZEN_FF, VEROZEN_SIDE, VEROZEN_RANK = 1536, 256, 16     # a token's experts together have the 12288 of Vemedra's feed-forward


def verozen_config(layers=VEROZEN_LAYERS):
    """The widths and heads of ``vemedra_config``: of every four layers two gated linear attention, one sigmoid attention, one
    retention."""
    mlp = {"kind": "moe", "expert": {"ff": VEROZEN_FF}, "router": VEROZEN_EXPERTS}
    gla = {"type": "gla", "mlp": mlp, "mixer": {"heads": 16, "dim": 128, "vdim": 256, "tau": 16.0, "rank": VEROZEN_RANK}}
    att = {"type": "attention", "mlp": mlp, "mixer": {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": {"base": 1e6, "dims": 128}}}
    ret = {"type": "retention", "mlp": mlp, "mixer": {"heads": 16, "dim": 128, "vdim": 256, "decay": [1 - 2.0 ** -(5 + 0.5 * h) for h in range(16)],
                                                      "rot": {"base": 1e4, "dims": 128}}}
    return {"architecture": "Verozen", "vocab": 151936, "width": 4096, "norm": {"eps": 1e-6, "groups": 4}, "postln_alpha": 2.0,
            "token_side": {"dim": VEROZEN_SIDE}, "layers": [(gla, gla, att, ret)[i % 4] for i in range(layers)]}


def verozen_kernels(dev, peaks, T=8192, context=2048):
    """Each kernel of a Verozen layer on its own, on inputs larger than L2 (rotating copies), against its roofline, beside
    the like kernel of a Vemedra layer."""
    from nanoquantization_b200 import _lib
    from nanoquantization_b200.engine import StepBatch
    from nanoquantization_b200.layers import mixers as ops, moe
    from nanoquantization_b200.layers.sequence_mixers import AttentionMixer, GatedLinearMixer, RetentionMixer, SigmoidAttentionMixer
    hbm, bf16 = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    W, H, G, D, RH, RD, RV, FF, bs = 4096, 32, 8, 128, 16, 128, 256, 12288, 256
    E, top, ff, n_side, rank = VEROZEN_EXPERTS["experts"], VEROZEN_EXPERTS["top"], VEROZEN_FF, VEROZEN_SIDE, VEROZEN_RANK
    rows, dt, f32 = [], torch.bfloat16, torch.float32

    def rnd(*shape, dtype=dt):
        return torch.randn(*shape, device=dev, dtype=f32).to(dtype)

    def add(phase, name, us, nbytes=0, flops=0):
        tb, tf = nbytes / hbm * 1e6, flops / bf16 * 1e6
        rows.append({"phase": phase, "kernel": name, "us": round(us, 2), "bound": "hbm" if tb >= tf else "tensor",
                     "of_roofline": round(max(tb, tf) / us, 3)})

    def step(n, B, start):
        blocks = -(-(start + n) // bs)
        return StepBatch.host([[0] * n] * B, [start] * B, [[b * blocks + i for i in range(blocks)] for b in range(B)], list(range(B)), blocks, bs).to(dev)
    sig = SigmoidAttentionMixer(heads=H, kv_heads=G, dim=D, rot_base=1e6, rot_dims=D, interleaved=True, scale=D ** -0.5, eps=1e-6, device=dev)
    for t in (sig.q_norm, sig.k_norm, sig.temp):
        t.fill_(1.0)
    sig.bias.fill_(-7.0)
    cap = AttentionMixer(heads=H, kv_heads=G, dim=D, vdim=D, chunk=T, rot_base=1e6, rot_dims=D, scale=D ** -0.5, softcap=50.0, device=dev)
    gla = GatedLinearMixer(heads=RH, dim=RD, vdim=RV, rank=rank, tau=16.0, eps=1e-6, dtype=dt, device=dev)
    gla.a2.copy_(rnd(RH * RD, rank) * rank ** -0.5)
    gla.a2_bias.copy_(2 + rnd(RH * RD, dtype=f32))
    gla.norm.fill_(1.0)
    decay = [1 - 2.0 ** -(5 + 0.5 * h) for h in range(RH)]
    ret = RetentionMixer(heads=RH, dim=RD, vdim=RV, decay=decay, eps=1e-6, rot_base=1e4, rot_dims=RD, device=dev)
    plain = RetentionMixer(heads=RH, dim=RD, vdim=RV, decay=decay, eps=1e-6, device=dev)
    router = _lib.RouterDesc(E, top, VEROZEN_EXPERTS["groups"]["count"], VEROZEN_EXPERTS["groups"]["keep"], 2.5, None)
    lin_cols = 2 * RH * RD + 2 * RH * RV
    # prefill
    one = step(T, 1, 0)
    x, nw, cw = [rnd(T, W, dtype=f32) for _ in range(2)], torch.ones(W, device=dev), rnd(4, W, dtype=f32)
    cst = torch.zeros(65, 3, W, device=dev)
    add("prefill", "norm in 4 groups after the sum", _device_us(lambda i: ops.post_norm_(x[i % 2], None, 1.0, nw, 4, 1e-6, dt), 8), T * W * 10)
    y8 = [rnd(T, top, W) for _ in range(2)]
    add("prefill", "the same with the sum of 8 experts", _device_us(lambda i: ops.post_norm_(x[i % 2], y8[i % 2], 2.0, nw, 4, 1e-6, dt), 8), T * W * (10 + 2 * top))
    del y8
    yf = [rnd(T, W, dtype=f32) for _ in range(2)]
    add("prefill", "side input: norm and add", _device_us(lambda i: ops.add_normed_(x[i % 2], yf[i % 2], nw, 1e-6, dt), 8), T * W * 14)
    del yf
    add("prefill", "Vemedra: rmsnorm + convolution", _device_us(lambda i: ops.rmsnorm_conv(x[i % 2], nw, cw, cst, one, 1e-6, dt), 8), T * W * 6)
    pq = [rnd(T, (H + 2 * G) * D) for _ in range(3)]
    kc, vc = rnd(T // bs + 1, bs, G, D), rnd(T // bs + 1, bs, G, D)
    rd, rr = sig.rope_desc(), ret.rope_desc()
    add("prefill", "head norm + rotary + K/V store", _device_us(lambda i: ops.norm_rope(pq[i % 3], kc, vc, rd, one, 0, H * D, H * D), 9), T * (2 * H * D + 3 * G * D) * 2)
    add("prefill", "Vemedra: rotary + K/V store", _device_us(lambda i: ops.rope_store(pq[i % 3], kc, vc, cap.inv_freq, one, 0, H * D, (H + G) * D, H), 9),
        T * (2 * H * D + 4 * G * D) * 2)
    o = rnd(T, H * D)
    for name, m in (("sigmoid attention", sig), ("Vemedra: capped softmax attention, one chunk of all", cap)):
        d = m.desc()
        us = _device_us(lambda i: ops.chunk_attention(pq[i % 3][:, :H * D], kc, vc, o, d, one), 4)
        add("prefill", name, us, flops=T * T / 2 * 4 * D * H)
    del pq, o
    pl, act, st = [rnd(T, lin_cols + rank) for _ in range(2)], rnd(T, RH * RV), torch.zeros(65, RH, RD, RV, device=dev)
    gd = plain.desc()
    flow = T * (2 * RH * RD + 3 * RH * RV) * 2
    add("prefill", "gated linear attention + norm + gate (4 launches)", _device_us(lambda i: ops.gla_gated(pl[i % 2], 0, gla, st, act, 0, one), 4), flow + T * rank * 2,
        4 * T * RH * RD * RV)
    add("prefill", "rotary of retention", _device_us(lambda i: ops.norm_rope(pl[i % 2], None, None, rr, one, 0, RH * RD, 0), 8), T * 4 * RH * RD * 2)
    add("prefill", "retention + norm + gate (3 launches, as Vemedra's)", _device_us(lambda i: ops.retention_gated(pl[i % 2], 0, gd, plain.decay, st, act, 0, one), 4), flow,
        4 * T * RH * RD * RV)
    del pl, act
    h = [rnd(T, W) for _ in range(2)]
    up, down, wr = rnd(E, ff, W), rnd(E, W, ff), rnd(E, W)
    plan = moe.route(rnd(T, E, dtype=f32), router)
    u = moe.experts_up(h[0], up, plan)
    lg = [rnd(T, E, dtype=f32) for _ in range(2)]
    add("prefill", "router product (library)", _device_us(lambda i: ops.linear(h[i % 2], wr, f32), 8), T * (W * 2 + E * 4) + E * W * 2)
    add("prefill", "routing and sort (3 launches)", _device_us(lambda i: moe.route(lg[i % 2], router), 8), T * (E * 4 + top * 16))
    add("prefill", "experts' first product + gelu", _device_us(lambda i: moe.experts_up(h[i % 2], up, plan), 4), flops=2 * T * top * W * ff)
    add("prefill", "experts' second product + weight", _device_us(lambda i: moe.experts_down(u, down, plan), 4), flops=2 * T * top * W * ff)
    del u
    w2, y = rnd(W, FF), rnd(T, FF)
    add("prefill", "Vemedra: down product + residual (library)", _device_us(lambda i: ops.linear_residual_(x[i % 2], y, w2), 4), flops=2 * T * W * FF)
    del w2, y
    ids, table = torch.randint(0, 1000, (T,), device=dev), rnd(1000, 8 * n_side)
    sg, sp = rnd(n_side, W), rnd(W, n_side)
    add("prefill", "side input: gate product (library) + gelu + table", _device_us(lambda i: ops.linear_gelu_table(h[i % 2], sg, ids, table, n_side), 8),
        T * (W + n_side) * 2, 2 * T * W * n_side)
    gg = [rnd(T, n_side) for _ in range(2)]
    add("prefill", "side input: product (library)", _device_us(lambda i: ops.linear(gg[i % 2], sp, f32), 8), T * (n_side * 2 + W * 4), 2 * T * W * n_side)
    del x, h, lg, gg
    torch.cuda.empty_cache()
    # decode: weights and caches rotate over copies larger than L2
    for B in (1, 16):
        ph, s, h = f"decode, batch {B}", step(1, B, context - 1), rnd(B, W)
        stream, nin = rnd(B, W, dtype=f32), lin_cols + rank
        ws = [rnd(nin, W) for _ in range(3)]
        add(ph, "merged input product (gated linear attention)", _device_us(lambda i: ops.linear(h, ws[i % 3]), 12), nin * W * 2)
        ws = [rnd(W, RH * RV) for _ in range(8)]
        a4 = rnd(B, RH * RV)
        add(ph, "output product + scaled residual", _device_us(lambda i: ops.linear_residual_(stream, a4, ws[i % 8], 2.0), 16), W * RH * RV * 2)
        # disjoint experts from call to call, as far as there are
        plans, bytes_ = [], []
        for c in range(4):
            lg = rnd(B, E, dtype=f32)
            if B == 1:
                lg[:, 8 * c:8 * c + 8] += 20
            plans.append(moe.route(lg, _lib.RouterDesc(E, top, 1, 1, 1.0, None)))
            bytes_.append(int(plans[-1].active[0]) * ff * W * 2)
        us_ = [moe.experts_up(h, up, p) for p in plans]
        add(ph, "experts' first product + gelu", _device_us(lambda i: moe.experts_up(h, up, plans[i % 4]), 12), sum(bytes_) / 4)
        add(ph, "experts' second product + weight", _device_us(lambda i: moe.experts_down(us_[i % 4], down, plans[i % 4]), 12), sum(bytes_) / 4)
        ws = [rnd(2 * FF, W) for _ in range(2)]
        add(ph, "Vemedra: gate | up product + clamped GLU", _device_us(lambda i: ops.dense_glu(h, ws[i % 2], 7.0), 8), 2 * FF * W * 2)
        ws, f12 = [rnd(W, FF) for _ in range(3)], rnd(B, FF)
        add(ph, "Vemedra: down product + residual", _device_us(lambda i: ops.linear_residual_(stream, f12, ws[i % 3]), 12), FF * W * 2)
        ws = [rnd(E, W) for _ in range(2)]
        add(ph, "router product", _device_us(lambda i: ops.linear(h, ws[i % 2], f32), 16), E * W * 2)
        lg = rnd(B, E, dtype=f32)
        add(ph, "routing and sort", _device_us(lambda i: moe.route(lg, router), 16), B * E * 4)
        idb = torch.randint(0, 1000, (B,), device=dev)
        add(ph, "side input: gate product + gelu + table", _device_us(lambda i: ops.linear_gelu_table(h, sg, idb, table, n_side), 16), n_side * W * 2)
        gb = rnd(B, n_side)
        add(ph, "side input: product", _device_us(lambda i: ops.linear(gb, sp, f32), 16), n_side * W * 2)
        yb, y8 = rnd(B, W, dtype=f32), rnd(B, top, W, dtype=f32)
        add(ph, "side input: norm and add", _device_us(lambda i: ops.add_normed_(stream, yb, nw, 1e-6, dt), 16), B * W * 14)
        add(ph, "norm in 4 groups after the sum", _device_us(lambda i: ops.post_norm_(stream, None, 1.0, nw, 4, 1e-6, dt), 16), B * W * 10)
        add(ph, "the same with the sum of 8 experts", _device_us(lambda i: ops.post_norm_(stream, y8, 2.0, nw, 4, 1e-6, dt), 16), B * W * (10 + 4 * top))
        add(ph, "Vemedra: rmsnorm + convolution", _device_us(lambda i: ops.rmsnorm_conv(stream, nw, cw, cst, s, 1e-6, dt), 16), B * W * (6 + 24) + W * 20)
        del ws
        n = 8 if B == 1 else 2   # copies of cache and state
        copies = []
        for _ in range(n):
            nb = B * (context // bs)
            copies.append((rnd(nb, bs, G, D), rnd(nb, bs, G, D), torch.zeros(B, RH, RD, RV, device=dev)))
        pa, pl, ac = rnd(B, (H + 2 * G) * D), rnd(B, lin_cols + rank), rnd(B, H * D)
        kv_bytes, st_bytes = B * context * 2 * G * D * 2, 2 * B * RH * RD * RV * 4
        for name, m in (("head norm + rotary + store + sigmoid attention", sig), ("Vemedra: rotary + store + attention", cap)):
            d, r = m.desc(), m.rope_desc()
            v = m.value_column(0)
            add(ph, name, _device_us(lambda i: ops.mixer_decode(pa, ac, (d, r, 0, v, 0, copies[i % n][0], copies[i % n][1]), None, s), 2 * n), kv_bytes)
        for name, m in (("gated linear attention + norm + gate", gla), ("rotary + retention + norm + gate", ret), ("Vemedra: retention + norm + gate", plain)):
            d = m.desc()
            add(ph, name, _device_us(lambda i: ops.mixer_decode(pl, ac, None, (d, 0, 0, copies[i % n][2]), s), 2 * n), st_bytes)
        del copies
    return rows


def run_verozen(args):
    """--verozen: random-init layers of real sizes through the engine, beside Vemedra layers of the same width, heads and
    (active) feed-forward, and every kernel against its roofline."""
    from nanoquantization_b200.engine import LLMEngine
    from nanoquantization_b200.models import VemedraConfig, VemedraForCausalLM, VerozenConfig, VerozenForCausalLM
    torch.cuda.set_device(0)
    dev, dt = torch.device("cuda", 0), torch.bfloat16
    torch.manual_seed(0)
    with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as fh:
        peaks = json.load(fh)
    line = {"what": "Verozen beside Vemedra, random init, one GPU, bf16", "layers": VEROZEN_LAYERS,
            "note": "weights and caches larger than L2; rooflines are the measured copy bandwidth and bf16 peak"}
    sampler = ClockSampler(0)
    sampler.start()
    if not args.verozen_kernels_only:
        for name, build in (("verozen", lambda: VerozenForCausalLM(VerozenConfig.from_dict(verozen_config()), device=dev, dtype=dt)),
                            ("vemedra", lambda: VemedraForCausalLM(VemedraConfig.from_dict(vemedra_config()), device=dev, dtype=dt))):
            model = build()
            for key, t in model.checkpoint_tensors().items():
                if "norm" in key or key.endswith("temp"):
                    t.fill_(1.0)
                elif key.endswith("pb"):
                    t.fill_(-7.0)
                else:
                    t.copy_(torch.randn(t.shape, device=dev) * (t.shape[-1] ** -0.5 if t.dim() > 1 else 0.1))
            eng = LLMEngine(model, num_blocks=64 * 9 + 40, max_batch=64)
            line[name] = _engine_throughput(eng, 151936, (1, 16, 64), 2047, 8192)
            line[name]["weights_gb"] = round(sum(t.numel() * t.element_size() for t in model.buffers()) / 1e9, 2)
            del eng, model
            torch.cuda.empty_cache()
    line["kernels"] = verozen_kernels(dev, peaks)
    line["clocks"] = sampler.stop()
    emit(json.dumps(line))


# --------------------------------------------------------------------------
# checker legs of our arm (after the timed regions)
# --------------------------------------------------------------------------
def reference_gpu_leg(layers, xs_dev, points, per_point, dev):
    """The reference's own WQLinear_GEMM.forward on this GPU, on the same packed tensors and activations:
    its fused Triton kernel below 256 tokens (gemm.py:563-564), its Triton dequantise kernel followed by
    torch.matmul from 256 tokens (gemm.py:558-561).  Unmodified code imported from baseline/_ref; only
    the benchmark's shapes (N % 256 == 0, K % 32 == 0), for which its kernels' edge masks are not reached.
    Per point: microseconds (same rotation over weight copies, replayed as a CUDA graph when the reference
    can be captured) and the output's distance from ours."""
    ref_root = os.path.join(ROOT, "baseline", "_ref")
    if not os.path.isdir(os.path.join(ref_root, "nanoquantization")):
        return {"unavailable": "baseline/_ref holds no install of the reference"}
    try:
        sys.path.insert(0, ref_root)
        from nanoquantization.layers.gemm import WQLinear_GEMM as RefLinear
    except Exception as exc:
        return {"unavailable": f"import of the reference failed: {type(exc).__name__}: {exc}"[:300]}
    finally:
        if ref_root in sys.path:
            sys.path.remove(ref_root)
    out, ours_us = [], {(p["M"], p["K"], p["N"]): p["us"] for p in per_point}
    try:
        refs = {}
        for si, copies in layers.items():
            refs[si] = []
            for lin in copies:
                r = RefLinear(4, GROUP, lin.in_features, lin.out_features, dev, False, lin.qscales.dtype)
                r.qweight, r.qscales, r.qzeros = lin.qweight, lin.qscales, lin.qzeros   # the same memory
                refs[si].append(r)
        graphs = 0
        for (si, M) in points:
            K, N, _ = SHAPES[si]
            x = xs_dev[(si, M)]
            copies = refs[si]
            reps = max(8, 2 * len(copies)) if M <= 128 else 4
            y_ref = copies[0](x)              # compiles the Triton kernels on first use
            y_ours = layers[si][0](x)
            torch.cuda.synchronize()
            err = float((y_ref.float() - y_ours.float()).abs().max() / y_ref.float().abs().max())

            def burst(copies=copies, x=x, reps=reps):
                for r in range(reps):
                    copies[r % len(copies)](x)
            fn, graphed = burst, False
            try:
                side = torch.cuda.Stream()
                side.wait_stream(torch.cuda.current_stream())
                with torch.cuda.stream(side):
                    burst()
                torch.cuda.current_stream().wait_stream(side)
                torch.cuda.synchronize()
                g = torch.cuda.CUDAGraph()
                with torch.cuda.graph(g):
                    burst()
                fn, graphed = g.replay, True
                graphs += 1
            except Exception:
                torch.cuda.synchronize()
            for _ in range(2):
                fn()
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            us = e0.elapsed_time(e1) * 1e3 / reps
            mine = ours_us[(M, K, N)]
            out.append({"M": M, "K": K, "N": N, "us": round(us, 2), "ours_us": mine, "speedup": round(us / mine, 2),
                        "rel_err_vs_ours": float(f"{err:.3e}"), "graph": graphed})
            del fn, g
            torch.cuda.empty_cache()
    except Exception as exc:
        torch.cuda.synchronize()
        return {"unavailable": f"the reference did not run on this GPU: {type(exc).__name__}: {exc}"[:400],
                "points_done": out}
    total_ref, total_ours = sum(p["us"] for p in out), sum(p["ours_us"] for p in out)
    small = [p for p in out if p["M"] <= 16]
    return {"what": "reference WQLinear_GEMM.forward (Triton kernels JIT-compiled here, torch.matmul from 256 tokens), "
                    "unmodified, from baseline/_ref; same tensors, per-point bursts over rotating weight copies",
            "sweep_us": round(total_ref, 1), "ours_sweep_us": round(total_ours, 1),
            "speedup_sweep": round(total_ref / total_ours, 2),
            "speedup_decode_points": round(sum(p["us"] for p in small) / sum(p["ours_us"] for p in small), 2),
            "max_rel_err_vs_ours": max(p["rel_err_vs_ours"] for p in out),
            "graphed_points": graphs, "points": out}


def tp_parity_leg(world, rank, dev, dtype, comm):
    """Correctness of the tensor-parallel path on the GPUs of this run: one column-parallel and one
    row-parallel shape of the sweep at 1, 16 and 128 tokens.  Every rank builds the same full tensors from
    a seed and loads its shard; the gathered column-parallel result and the all-reduced row-parallel result
    (through NCCL, and through the peer-memory path when there is one) are compared with the CPU oracle on
    the full tensors, the peer path must give the same bits on every rank and on every repetition, and
    the peer communicator must have recorded no give-up."""
    import torch.distributed as dist
    import nanoquantization_b200 as nq
    from oracle import awq_oracle as O
    res = {"points": 0, "max_rel_err": 0.0, "peer_bits_equal_across_ranks": True, "peer_repeatable": True,
           "nccl_equals_peer_bits": True, "bound": 2e-3}
    for (K, N, kind) in ((4096, 12288, "column"), (12288, 4096, "row")):
        g = torch.Generator().manual_seed(K + N)
        qw = torch.randint(-2 ** 31, 2 ** 31, (K, N // 8), generator=g, dtype=torch.int64).to(torch.int32)
        qz = torch.randint(-2 ** 31, 2 ** 31, (K // GROUP, N // 8), generator=g, dtype=torch.int64).to(torch.int32)
        qs = (torch.rand(K // GROUP, N, generator=g) * 9e-3 + 1e-3).to(dtype)
        x_all = torch.randn(128, K, generator=g).to(dtype)
        W = O.dequantize(qw, qs, qz).float() if rank == 0 else None
        if kind == "column":
            lin = nq.ColumnParallelWQLinear(4, GROUP, K, N, world, rank, dev, False, dtype, gather_output=True)
        else:
            lin = nq.RowParallelWQLinear(4, GROUP, K, N, world, rank, dev, False, dtype)
        lin.load_full(qw.to(dev), qs.to(dev), qz.to(dev))
        for M in (1, 16, 128):
            x = x_all[:M].to(dev)
            xin = lin.input_slice(x).contiguous() if kind == "row" else x
            ys = [("nccl", lin(xin))]
            if kind == "row" and comm is not None:
                lin.attach_comm(comm)
                y1 = lin(xin)
                y2 = lin(xin)
                lin.attach_comm(None)
                res["peer_repeatable"] &= bool(torch.equal(y1, y2))
                parts = [torch.empty_like(y1) for _ in range(world)]
                dist.all_gather(parts, y1)
                res["peer_bits_equal_across_ranks"] &= all(bool(torch.equal(p_, y1)) for p_ in parts)
                res["nccl_equals_peer_bits"] &= bool(torch.equal(y1, ys[0][1]))
                ys.append(("peer", y1))
            torch.cuda.synchronize()
            if rank == 0:
                ref = x_all[:M].float() @ W
                for _name, y in ys:
                    res["max_rel_err"] = max(res["max_rel_err"], O.rel_err(y, ref))
            res["points"] += len(ys)
        del lin
    flags = torch.tensor([int(res["peer_bits_equal_across_ranks"]), int(res["peer_repeatable"]),
                          int(res["nccl_equals_peer_bits"])], device=dev)
    dist.all_reduce(flags, op=dist.ReduceOp.MIN)
    res["peer_bits_equal_across_ranks"], res["peer_repeatable"], res["nccl_equals_peer_bits"] = (bool(v) for v in flags.tolist())
    res["peer_allreduce_status"] = comm.status() if comm is not None else None
    res["max_rel_err"] = float(f"{res['max_rel_err']:.3e}")
    res["ok"] = bool(res["max_rel_err"] <= res["bound"] and res["peer_bits_equal_across_ranks"] and res["peer_repeatable"]
                     and not res["peer_allreduce_status"]) if rank == 0 else None
    res["note"] = ("nccl_equals_peer_bits is reported, not required: NCCL adds the ranks' 16-bit partial results in its "
                   "own order and precision, the peer path adds them in rank order in fp32 and rounds once")
    return res


# --------------------------------------------------------------------------
# CPU arm: the restatement of the reference arithmetic on the host cores
# --------------------------------------------------------------------------
class CpuSweep:
    """The 30 points on the host: per point, unpack by shifts and (q - z) * s into the 16-bit weight (what
    the reference's forward does on every call, gemm.py:558-564), then the matmul in fp32.  Weights are made
    once per shape (uniform random words = uniform int4 values)."""

    def __init__(self):
        self.shapes = {}
        for si, (K, N, _kind) in enumerate(SHAPES):
            g = torch.Generator().manual_seed(100 + si)
            self.shapes[si] = (
                torch.randint(-2 ** 31, 2 ** 31, (K, N // 8), generator=g, dtype=torch.int64).to(torch.int32),
                (torch.rand(K // GROUP, N, generator=g) * 9e-3 + 1e-3).to(torch.float16),
                torch.randint(-2 ** 31, 2 ** 31, (K // GROUP, N // 8), generator=g, dtype=torch.int64).to(torch.int32))
        self.xs = {}
        for si, (K, N, _kind) in enumerate(SHAPES):
            g = torch.Generator().manual_seed(200 + si)
            big = torch.randn(max(MS), K, generator=g).to(torch.float16)
            for M in MS:
                self.xs[(si, M)] = big[:M]

    def run_pass(self):
        """One pass over all points; returns (seconds, per-point seconds)."""
        from oracle import awq_oracle as O
        per = []
        t_all = time.perf_counter()
        for M in MS:
            for si, (K, N, _kind) in enumerate(SHAPES):
                qw, qs, qz = self.shapes[si]
                t0 = time.perf_counter()
                W = O.dequantize_threaded(qw, qs, qz).float()
                y = self.xs[(si, M)].float() @ W
                per.append({"M": M, "K": K, "N": N, "ms": round((time.perf_counter() - t0) * 1e3, 2)})
                del W, y
        return time.perf_counter() - t_all, per


def cpu_baseline():
    cores = os.cpu_count() or 1
    torch.set_num_threads(cores)
    sweep = CpuSweep()
    secs, per = sweep.run_pass()
    return {"value": round(secs * 1e6, 1), "unit": "us", "cores": cores, "kind": "port",
            "sample": ("one real pass over all 30 points of the sweep by the CPU restatement (unpack by shifts, (q-z)*s, "
                       "fp32 matmul; torch and numpy on all host threads), nothing extrapolated"),
            "wall_s": round(secs, 1), "points": per}


def run_reference(args):
    rank = int(os.environ.get("RANK", "0"))
    if rank != 0:
        return
    cores = os.cpu_count() or 1
    torch.set_num_threads(cores)
    steps, warm = args.steps, args.warmup
    sweep = CpuSweep()
    t_start = time.perf_counter()
    budget_s = args.reference_budget
    warm_done = 0
    for _ in range(min(warm, 1)):       # one pass warms the allocator and the thread pools; more would only cost minutes
        sweep.run_pass()
        warm_done += 1
    passes, per = [], None
    for i in range(steps):
        if passes and (time.perf_counter() - t_start) + passes[-1] > budget_s:
            break                        # a pass takes about 12 s: stop where the next one would pass the wall budget
        secs, per = sweep.run_pass()
        passes.append(secs)
    us = sum(passes) / len(passes) * 1e6
    sample = (f"{len(passes)} real passes over all 30 points by the CPU restatement of the reference arithmetic (unpack by shifts, "
              f"(q-z)*s, fp32 matmul; torch and numpy on all {cores} host threads), nothing extrapolated; {warm_done} warm-up pass")
    line = {"impl": "reference", "metric": "w4a16_gemm_sweep_us", "value": round(us, 1), "unit": "us",
            "n_gpus": args.gpus, "steps": len(passes), "steps_requested": steps, "steps_measured": len(passes),
            "warmup": warm_done, "ms_per_step": round(us / 1e3, 3),
            "higher_is_better": False, "scaling": "strong", "vs_baseline": None,
            "dtype": "f32", "data": "synthetic",
            "config": sweep_config("host cores", "CPU restatement, one call per point"),
            "cpu_baseline": {"value": round(us, 1), "unit": "us", "cores": cores, "kind": "port", "sample": sample},
            "e2e": {"value": round(us, 1), "unit": "us", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
            "gpu_launches": 0, "wall_s": round(time.perf_counter() - t_start, 1), "points": per}
    emit(json.dumps(line))


def run_serve(args):
    import torch.distributed as dist
    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    torch.cuda.set_device(local)
    dev = torch.device("cuda", local)
    if world > 1:
        if os.environ.get("NCCL_DEBUG", "VERSION").upper() == "VERSION":
            os.environ["NCCL_DEBUG"] = "WARN"
        dist.init_process_group("nccl", device_id=dev)
    dtype = torch.bfloat16 if args.dtype == "bf16" else torch.float16
    out = serve_bench(world, rank, dev, dtype, requests=args.requests, arch=args.serve)
    if rank == 0:
        emit(json.dumps(out))
    leave_distributed(world)


def run_point(args):
    """One (M, K, N) point launched --reps times over rotating weight copies, timed with CUDA
    events; the small, single-kernel case profilers are pointed at."""
    import nanoquantization_b200 as nq  # noqa: F401
    from nanoquantization_b200 import _lib
    M, K, N = (int(v) for v in args.point.split(","))
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    dtype = torch.bfloat16 if args.dtype == "bf16" else torch.float16
    ncopy = max(2, -(-int(1.5 * L2_BYTES) // weight_bytes(K, N)))
    layers = [make_layer(K, N, 7 + c, dev, dtype) for c in range(ncopy)]
    x = torch.randn(M, K, device=dev).to(dtype)
    def burst():
        for r in range(args.reps):
            layers[r % ncopy](x)
    burst()
    torch.cuda.synchronize()
    fn = burst
    if not args.no_graph:  # replayed as one CUDA graph so that the number is device time, not Python launch time
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            burst()
        fn = graph.replay
        fn()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    fn()
    e1.record()
    torch.cuda.synchronize()
    _lib.check_workspaces()
    us = e0.elapsed_time(e1) * 1e3 / args.reps
    emit(json.dumps({"point": [M, K, N], "reps": args.reps, "us_per_call_incl_launch": round(us, 2),
                      "kernel": _lib.load().nqb200_gemm_kernel_name(M, N, K, GROUP, 0).decode()}))


_REAL_STDOUT = None


def protect_stdout():
    """Libraries (NCCL's version banner, for one) print to stdout; the contract is ONE JSON line
    there.  Everything written to fd 1 from here on goes to stderr; emit() writes to the real stdout."""
    global _REAL_STDOUT
    sys.stdout.flush()
    _REAL_STDOUT = os.dup(1)
    os.dup2(2, 1)


def emit(text: str) -> None:
    if _REAL_STDOUT is None:
        print(text, flush=True)
    else:
        os.write(_REAL_STDOUT, (text + "\n").encode())


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=10)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--no-decode", action="store_true", help="skip the Qwen3-8B decode tokens/s section")
    ap.add_argument("--no-reference-gpu", action="store_true", help="skip the reference's own GPU path (1 GPU)")
    ap.add_argument("--no-serve", action="store_true", help="with --gpus 8: skip the Qwen3-32B continuous-batching workload")
    ap.add_argument("--serve-budget", type=int, default=240, help="seconds the --gpus 8 serving workload may take before the line is printed without it")
    ap.add_argument("--max-seconds", type=int, default=840, help="a multi-GPU run that has not finished by then prints an `unavailable` line and leaves")
    ap.add_argument("--nccl-only", action="store_true", help="tensor parallel: all-reduce through NCCL only")
    ap.add_argument("--reference-budget", type=float, default=330.0,
                    help="--impl reference: wall-clock seconds after which no further pass is started")
    ap.add_argument("--point", default=None, help="M,K,N: run only this point (for profilers)")
    ap.add_argument("--reps", type=int, default=6)
    ap.add_argument("--no-graph", action="store_true", help="with --point: plain launches (what a profiler should see)")
    ap.add_argument("--dtype", default="f16", choices=["f16", "bf16"])
    ap.add_argument("--serve", nargs="?", const="qwen3-32b", default=None,
                    help="instead of the sweep: the continuous-batching workload on this architecture (tensor-parallel under torchrun)")
    ap.add_argument("--vemedra", action="store_true",
                    help="instead of the sweep: Vemedra layers of real sizes beside Qwen3 layers of the same size, and every kernel against its roofline")
    ap.add_argument("--vemedra-kernels-only", action="store_true", help="with --vemedra: the kernels alone")
    ap.add_argument("--verozen", action="store_true",
                    help="instead of the sweep: Verozen layers of real sizes beside Vemedra layers of the same size, and every kernel against its roofline")
    ap.add_argument("--verozen-kernels-only", action="store_true", help="with --verozen: the kernels alone")
    ap.add_argument("--requests", type=int, default=256)
    ap.add_argument("--decode-only", type=int, default=0, metavar="BATCH",
                    help="only the Qwen3-8B decode point of this batch size, 1 GPU (the case a launch list is taken of)")
    args = ap.parse_args()
    protect_stdout()
    if args.decode_only:
        torch.cuda.set_device(0)
        dtype = torch.bfloat16 if args.dtype == "bf16" else torch.float16
        emit(json.dumps(decode_bench(1, 0, torch.device("cuda", 0), dtype, batches=(args.decode_only,), steps=4, prefill=False)))
    elif args.vemedra:
        run_vemedra(args)
    elif args.verozen:
        run_verozen(args)
    elif args.serve:
        run_serve(args)
    elif args.point:
        run_point(args)
    elif args.impl == "reference":
        run_reference(args)
    else:
        run_ours(args)


if __name__ == "__main__":
    main()
