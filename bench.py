#!/usr/bin/env python
"""Headline benchmark: 27B-shape W4A16 decode (1 request) + prefill, 35B-A3B-shape MoE prefill.

    python bench.py --gpus N --steps K --warmup W

One JSON line on rank 0.  N = 1: ``value`` is decode tokens/s of one request on the 27B shape.  N > 1: ``value`` is
the decode tokens/s of ONE model sharded over the N GPUs (tensor parallel, fused NVLink kernels, 8 concurrent
requests): strong scaling, total work fixed as N grows.  Replica mode (a full copy per GPU) and the NCCL + cuBLAS
comparison are lines of ``extra``, next to the prompt-pass numbers.  Weights are random-init in the named
shapes and token ids are synthetic (no network for checkpoints or datasets).
Timing: CUDA events on the launching stream after W warm-up steps, bracketed by
a barrier and a device synchronize, max over ranks.  A decode step streams the
model's 12.7 GB of weights, far more than the 126 MB L2, so no L2 flush is
needed between steps ("inputs larger than L2").
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

BASELINE_DECODE_TPS = 164.0       # Qwen3.8-27B decode, 1 request, DFlash, 1x B70 (README.md:6,52)
BASELINE_PREFILL_TPS = 2800.0     # Qwen3.8-27B int8 prefill at 4k, 1x B70 (README.md:27)
BASELINE_MOE_PREFILL_TPS = 11223.0  # Ornith 35B-A3B prefill at 4k, 1x B70 (README.md:63)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""

    def __init__(self, gpu_index: int):
        self.idx = gpu_index
        self.proc = None
        self.lines = []

    def start(self):
        q = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--id={self.idx}", f"--query-gpu={q}",
                                          "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except Exception:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.lines.append(line.strip())

    def stop(self) -> dict:
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except Exception:
            pass
        sm, mx, reasons = [], None, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for ln in self.lines:
            f = [x.strip() for x in ln.split(",")]
            if len(f) < 7:
                continue
            try:
                sm.append(float(f[0])); mx = float(f[1])
            except ValueError:
                continue
            for n, v in zip(names, f[3:7]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        sm.sort()
        hi = [v for v in sm if v >= (sm[-1] * 0.5 if sm else 0)]   # samples under load
        med = hi[len(hi) // 2] if hi else None
        return {"sm_mhz": med, "sm_max_mhz": mx, "reasons": sorted(reasons), "samples": len(sm)}


def reference_arm(args):
    print(json.dumps({
        "impl": "reference",
        "unavailable": "reference is a C++26/Level Zero/OpenCL-C project for Intel Arc (needs the xe driver, "
                       "Level Zero loader and ocloc); it has no setup.py/pyproject, so pip cannot install it, "
                       "and it cannot build or run on an NVIDIA box",
    }))
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=4)
    ap.add_argument("--impl", default="b200")
    ap.add_argument("--model", default="dense-27b")
    ap.add_argument("--depth", type=int, default=4096, help="context length the decode steps run at")
    ap.add_argument("--prefill-len", type=int, default=4096)
    ap.add_argument("--what", default="all", help="decode | prefill | prefill32k | moe | w4 | spec | spec65k | batch32k | prefix | hybrid | mumusun | napadra | pefulorn | vogerax | tp | ep | pp | replica | all")
    ap.add_argument("--kv-cache", default="bf16")
    ap.add_argument("--int8-head", action="store_true")
    ap.add_argument("--prefill-backend", default="auto")
    ap.add_argument("--parallel", default="replica", help="replica | tp (N > 1)")
    ap.add_argument("--extras-budget-s", type=float, default=420.0, help="no further extra starts after this many seconds")
    ap.add_argument("--windows", type=int, default=5, help="timed windows of --steps steps; the median window is reported")
    ap.add_argument("--tp-rows", type=int, default=8, help="concurrent requests of the multi-GPU decode headline")
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm(args)

    import torch
    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    torch.cuda.set_device(local)
    dist = None
    ctl = None
    if world > 1:
        import datetime
        import torch.distributed as dist
        # a short collective timeout: a rank that left a section early must end the job, not hang the GPUs
        dist.init_process_group("nccl", device_id=torch.device("cuda", local), timeout=datetime.timedelta(minutes=4))
        ctl = dist.new_group(backend="gloo", timeout=datetime.timedelta(minutes=4))   # host-side agreement between sections

    from b200serve.utils.benchlib import run_decode_bench, run_prefill_bench
    from b200serve.ops import lib as K

    def barrier():
        if dist is not None:
            dist.barrier()
        torch.cuda.synchronize()

    sampler = ClockSampler(local)
    sampler.start()
    t_start = time.time()
    res = {}
    extra = {}
    state = {"multi_failed": False}

    def release():
        """Engines and their resident weight copies hold reference cycles: collect them before the next section."""
        import gc
        gc.collect()
        torch.cuda.empty_cache()

    def agree_failed(failed: bool) -> bool:
        """True on every rank if the section failed on any rank (host-side all-reduce, never queued behind GPU work)."""
        if ctl is None:
            return failed
        t = torch.tensor([1 if failed else 0], dtype=torch.int32)
        dist.all_reduce(t, op=dist.ReduceOp.MAX, group=ctl)
        return bool(int(t))

    def guarded(name, fn, multi_rank: bool = False):
        """A failing extra is recorded, never fatal: the headline line is printed regardless.  Extras that would start
        after the time budget is spent are skipped (the same decision on every rank: rank 0's clock is shared).
        After a section whose ranks talk to each other (``multi_rank``) the ranks agree on the outcome: if one of
        them raised, all record it and no further multi-rank section starts -- the ranks would meet in different
        collectives otherwise."""
        spent = time.time() - t_start
        if ctl is not None:
            t = torch.tensor([spent], dtype=torch.float64)
            dist.broadcast(t, src=0, group=ctl)
            spent = float(t)
        if spent > args.extras_budget_s:
            extra[name] = {"skipped": f"time budget of {args.extras_budget_s:.0f} s for extras was spent"}
            return None
        if multi_rank and state["multi_failed"]:
            extra[name] = {"skipped": "an earlier multi-rank section failed on some rank"}
            return None
        release()
        out, err = None, None
        try:
            out = fn()
        except Exception as e:  # noqa: BLE001
            err = f"{type(e).__name__}: {e}"[:400]
        if multi_rank and agree_failed(err is not None):
            state["multi_failed"] = True
            err = err or "another rank raised in this section"
        extra[name] = {"error": err} if err is not None else out
        release()
        return None if err is not None else out

    one_gpu_sections = world == 1 or args.what in ("decode", "prefill", "moe")
    if args.what in ("all", "decode") and one_gpu_sections:
        res = run_decode_bench(args, barrier)
        release()
    if args.what in ("all", "prefill") and one_gpu_sections:
        extra["prefill"] = run_prefill_bench(args, barrier, model=args.model, backend=args.prefill_backend)
        release()
        if args.what == "all":
            extra["prefill_int8"] = run_prefill_bench(args, barrier, model=args.model, backend="int8")
            release()
    if world == 1 and args.what in ("all", "prefill32k"):
        # the long prompt of the 27B configuration (32,768 tokens), both prompt-pass forms
        for name, backend in (("prefill_32k", args.prefill_backend), ("prefill_32k_int8", "int8")):
            guarded(name, lambda b=backend: run_prefill_bench(args, barrier, model=args.model, backend=b, n=32768, warm=1, reps=2))
    if args.what in ("all", "moe") and one_gpu_sections:
        extra["moe_prefill"] = run_prefill_bench(args, barrier, model="moe-35b-a3b", backend=args.prefill_backend)
        release()

        def moe_decode():
            # one request decoding on the 35B-A3B shape (3B active parameters per token), timed like the headline
            import copy
            a = copy.copy(args)
            a.model, a.windows = "moe-35b-a3b", 3
            r = run_decode_bench(a, barrier)
            return {"ms_per_step": r["ms_per_step"], "tokens_per_s": 1e3 / r["ms_per_step"],
                    "e2e_tokens_per_s": 1e3 / r["e2e_ms_per_step"], "depth": a.depth, "config": r["config"]}
        guarded("moe_decode", moe_decode)
    if world == 1 and args.what in ("mumusun", "napadra", "pefulorn", "vogerax"):
        # models that list their layers beside the closest other model at equal size (not part of "all")
        from b200serve.utils import bench_listed
        guarded(args.what, lambda: bench_listed.run(release, args.what))
    if world == 1 and args.what in ("all", "prefill", "moe", "w4"):
        # the prompt pass that keeps ONLY the int4 weights resident: the GEMM expands W4B blocks inside its shared-memory tiles
        if args.what != "moe":
            guarded("prefill_w4", lambda: run_prefill_bench(args, barrier, model=args.model, backend="w4"))
        if args.what != "prefill":
            guarded("moe_prefill_w4", lambda: run_prefill_bench(args, barrier, model="moe-35b-a3b", backend="w4"))

    def load_peaks():
        pk = os.path.join(os.path.dirname(os.path.abspath(__file__)), "MEASURED_PEAKS.json")
        if os.path.exists(pk):
            with open(pk) as f:
                return json.load(f)
        return {}

    def tp_headline():
        # ONE model over all the GPUs (tensor parallel, fused NVLink kernels), 8 concurrent requests: the whole job's
        # decode tokens/s, device-timed and end to end (host rows in, tokens out every step)
        from b200serve.models.config import preset
        from b200serve.parallel import tp as TP
        return TP.bench_decode(preset(args.model), "fused", args.depth, args.steps, max(args.warmup, 3), rows=args.tp_rows,
                               windows=args.windows, e2e=True, kv_dtype=args.kv_cache)

    def tp_extra():
        # the same group against the in-tree NCCL (+ cuBLAS for the prompt pass) build, the one-request step, the
        # prompt pass, the fused GEMM pair against its roofline, and a small sharded model against one GPU
        from b200serve.models.config import preset
        from b200serve.parallel import tp as TP
        from b200serve.parallel import tp_check as TPC
        cfg = preset(args.model)
        steps, warm = min(args.steps, 32), max(args.warmup, 3)
        tpx = {"world": world, "parallelism": f"tp{world}"}
        tpx["self_check_small_dense"] = TPC.self_check(TPC.widen_for(preset("small-dense"), world), ("fused", "nccl"), 200)
        tpx["spec_mtp_check_small_dense"] = TPC.spec_check(TPC.widen_for(preset("small-dense"), world), 200)
        tpx["decode8_nccl"] = TP.bench_decode(cfg, "nccl", args.depth, steps, warm, rows=args.tp_rows, kv_dtype=args.kv_cache)
        for mode in ("fused", "nccl"):
            tpx[f"decode_{mode}"] = TP.bench_decode(cfg, mode, args.depth, steps, warm)
            tpx[f"prefill_{mode}"] = TP.bench_prefill(cfg, mode, args.prefill_len)
        tpx["fused_ops"] = TP.bench_fused_ops(cfg, args.prefill_len, peaks=load_peaks())
        # speculative decoding under tensor parallelism: the MTP head sliced over the ranks, forced acceptance
        tpx["spec_mtp_k3_accept4_fused"] = TP.bench_spec_mtp(cfg, min(args.depth, 4096))
        # the 8-request serving case of the 27B configuration: 32,768-token prompts into an int8 KV cache, then the
        # eight requests decode together at that depth (the sharded model against itself on one GPU first)
        tpx["self_check_small_dense_int8kv"] = TPC.self_check(TPC.widen_for(preset("small-dense"), world), ("fused",), 200,
                                                              kv_dtype="int8")
        tpx["prefill_32k_int8kv_fused"] = TP.bench_prefill(cfg, "fused", 32768, reps=2, kv_dtype="int8")
        tpx["decode8_depth32k_int8kv_fused"] = TP.bench_decode(cfg, "fused", 32768, steps, warm, rows=args.tp_rows,
                                                               kv_dtype="int8")
        return tpx

    def replica_extra():
        # a full copy of the model per GPU, one request each (no collective involved): total tokens/s = N x one GPU
        r = run_decode_bench(args, barrier)
        t = torch.tensor([r["ms_per_step"]], device="cuda", dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        ms_max = float(t)
        return {"parallelism": f"replica x{world}", "ms_per_step_max_over_ranks": ms_max,
                "tokens_per_s_total": world * 1e3 / ms_max, "per_gpu_vs_baseline": (1e3 / ms_max) / BASELINE_DECODE_TPS,
                "config": r["config"]}

    def ep_extra():
        # the MoE shape with its experts spread over all the GPUs (data-parallel attention): fused dispatch /
        # return kernels against NCCL all-to-all around the same grouped GEMMs; a small model against one GPU first
        from b200serve.models.config import preset
        from b200serve.parallel import ep as EP
        from b200serve.parallel import ep_check as EPC
        out = {"world": world, "self_check_small_moe": EPC.self_check(preset("small-moe"))}
        out.update(EP.bench_prefill(preset("moe-35b-a3b"), args.prefill_len))
        # batched decode with the experts spread over the ranks: 16 requests over the group (the MoE configuration's batch)
        out["decode_batch16"] = EP.bench_decode_rows(preset("moe-35b-a3b"), max(16 // world, 1), args.depth,
                                                     min(args.steps, 32), max(args.warmup, 3))
        for total in (16384, 131072):     # the MoE configuration's prompt sizes, as totals over the group
            r = EP.bench_prefill(preset("moe-35b-a3b"), total // world, modes=("fused",), reps=2)
            out[f"prefill_fused_total_{total}"] = r["prefill_fused"]
        return out

    if world > 1 and args.what in ("all", "tp", "decode"):
        hd = guarded("tp_decode_headline", tp_headline, multi_rank=True)
        if hd is not None:
            res = {"metric": "decode_tokens_per_s", "baseline": 342.0,      # 8 requests, MTP, replica on 2 cards (README.md:6,51)
                   "ms_per_step": hd["ms_per_step"], "job_tokens_per_step": hd["rows"],
                   "e2e_ms_per_step": hd["e2e_ms_per_step"], "h2d": hd["h2d_bytes_per_step"], "d2h": hd["d2h_bytes_per_step"],
                   "launches": hd["launches_per_step"] * args.steps, "scaling": "strong",
                   "config": {"model": args.model, "global_batch": hd["rows"], "seq_len": args.depth,
                              "parallelism": f"tp{world}", "kv_cache": args.kv_cache, "lm_head": "bf16, vocabulary-parallel",
                              "weights": "W4A16 int4 g64, random init, sharded by heads / FFN columns",
                              "collectives": "fused NVLink kernels (peer stores + flags inside the GEMV / arg-max); no NCCL on the step",
                              "l2": "inputs larger than L2 (12.7 GB of weights per step over the group)",
                              "windows_ms_per_step": hd["windows_ms_per_step"]}}

    # The one-GPU features (speculation, prefix cache, hybrid model) are measured in one-GPU runs; a multi-GPU run
    # repeats them only when asked by name, so that its time goes to the scaling numbers and the fused collectives.
    if args.what == "spec" or (args.what == "all" and world == 1):
        from b200serve.utils.benchlib import run_spec_bench
        guarded("spec_forced_accept", lambda: run_spec_bench(args, barrier))
    if args.what == "spec65k" or (args.what == "all" and world == 1):
        from b200serve.utils.benchlib import run_spec_bench
        # the same loop behind a 65,536-token context (its prompt pass runs first, draft heads included)
        guarded("spec_after_65536", lambda: run_spec_bench(args, barrier, iters=8, depth=65536,
                                                           cases=(("mtp", 3, (3,), 0), ("dflash", 15, (7,), 0))))
    if args.what == "batch32k" or (args.what == "all" and world == 1):
        from b200serve.utils.benchlib import run_batch_after_long_prompt
        guarded("decode_8req_after_32k_int8kv", lambda: run_batch_after_long_prompt(args, barrier))
    if args.what == "prefix" or (args.what == "all" and world == 1):
        from b200serve.utils.benchlib import run_prefix_bench
        # every rank pins its own host store: a quarter of the prefix when several ranks share one host
        guarded("prefix_cache", lambda: run_prefix_bench(args, barrier, 65536 if world == 1 else 16384))
    if world == 1 and args.what in ("all", "hybrid"):
        from b200serve.utils.benchlib import run_hybrid_bench
        guarded("hybrid", lambda: run_hybrid_bench(args, barrier))
    if world > 1 and args.what in ("all", "tp"):
        guarded("tp", tp_extra, multi_rank=True)
    if world > 1 and args.what in ("all", "ep"):
        guarded("ep", ep_extra, multi_rank=True)
    if world == 2 and args.what in ("all", "pp"):
        def pp_extra():
            # the two GPUs as pipeline stages of one 27B model: the 32,768-token prompt pass and decode behind it
            from b200serve.models.config import preset
            from b200serve.parallel import pp as PP
            return PP.bench_pp(preset(args.model), 32768, min(args.steps, 32), max(args.warmup, 3))
        guarded("pp2", pp_extra, multi_rank=True)
    if world > 1 and args.what in ("all", "replica"):
        guarded("replica", replica_extra, multi_rank=True)
    clocks = sampler.stop()
    try:
        K.check_status()
    except Exception as e:  # noqa: BLE001
        extra["status"] = {"error": str(e)[:400]}

    def reduce_max(x: float) -> float:
        if dist is None:
            return x
        t = torch.tensor([x], device="cuda", dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        return float(t)

    if not res:   # no decode in this run: promote the first prompt-pass result (or, failing that, any timed extra)
        key = next((k for k, v in extra.items() if isinstance(v, dict) and "ms" in v and "baseline" in v), None)
        if key is not None:
            p = extra[key]
            res = {"ms_per_step": p["ms"], "tokens_per_step": p["tokens"], "e2e_ms_per_step": p.get("e2e_ms", p["ms"]),
                   "h2d": p.get("h2d", 0), "d2h": p.get("d2h", 0), "launches": p.get("launches", 0),
                   "metric": key + "_tokens_per_s", "baseline": p["baseline"], "config": p["config"]}
        else:
            res = {"ms_per_step": 0.0, "tokens_per_step": 0, "e2e_ms_per_step": 0.0, "h2d": 0, "d2h": 0,
                   "launches": 0, "metric": "extras_only", "baseline": None, "config": {"what": args.what}}
    ms = reduce_max(res["ms_per_step"])
    e2e_ms = reduce_max(res["e2e_ms_per_step"])
    # tokens of the WHOLE job per step: a sharded model emits its rows once; independent copies emit one row set each
    job_tokens = res["job_tokens_per_step"] if "job_tokens_per_step" in res else world * res["tokens_per_step"]
    value = job_tokens / (ms / 1e3) if ms else None
    e2e = job_tokens / (e2e_ms / 1e3) if e2e_ms else None
    if rank == 0:
        for k, p in extra.items():
            if "baseline" not in p:
                continue
            p["tokens_per_s"] = p["tokens"] / (p["ms"] / 1e3)
            p["vs_baseline"] = p["tokens_per_s"] / p["baseline"]
        out = {
            "metric": res.get("metric", "decode_tokens_per_s"),
            "value": value, "unit": "tokens/s", "n_gpus": world, "steps": args.steps, "warmup": args.warmup,
            "ms_per_step": ms, "higher_is_better": True, "scaling": res.get("scaling", "weak"),
            "vs_baseline": value / res["baseline"] if (value and res["baseline"]) else None,
            "vs_baseline_per_gpu": value / world / res["baseline"] if (value and res["baseline"]) else None,
            "dtype": "bf16",
            "dtype_detail": "W4A16: int4 g64 weights with fp16 group scales; bf16 activations, residual stream and KV; inside "
                            "the decode GEMV each 64-k group of a row's activations is re-quantised to 15-bit integers "
                            "(two int8 limbs, one fp32 scale) so the contraction runs as exact integer tensor-core sums; "
                            "fp32 accumulation across groups, bf16 lm_head",
            "data": "synthetic",
            "timing": f"median of {args.windows} windows of {args.steps} steps, each bracketed by barrier + synchronize, CUDA events, max over ranks",
            "config": res["config"],
            "clocks": clocks,
            "e2e": {"value": e2e, "unit": "tokens/s", "h2d_bytes_per_step": res["h2d"],
                    "d2h_bytes_per_step": res["d2h"]},
            "gpu_launches": res["launches"],
            "impl": "b200",
            "extra": extra,
        }
        print(json.dumps(out))
    if dist is not None:
        dist.barrier()
        dist.destroy_process_group()
    return 0


if __name__ == "__main__":
    sys.exit(main())
