#!/usr/bin/env python
"""Headline benchmark: GPT-2 124M BF16 training throughput (tokens/s), 16 sequences x 1024 tokens per
GPU, FP32-master AdamW + global-norm clip 1.0, fused shifted cross-entropy, synthetic uniform tokens,
random-init weights.  Weak scaling: per-GPU work is fixed; N > 1 shards optimizer state and
gradients over the data-parallel group (launched by torch.distributed.run, one rank per GPU).

  python bench.py --gpus N --steps K --warmup W          our implementation
  python bench.py --impl reference ...                   the unmodified reference's own single-GPU trainer,
                                                         built by baseline/build_ref.py (1 GPU only)

Prints ONE JSON line on rank 0.  `value` is the device-timed (CUDA events, max over ranks)
throughput of K optimizer steps with inputs resident on the device; `e2e` is the same metric through
the public trainer API including the pinned-host -> device copy of every step's tokens and the
device -> host read of its loss.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import tempfile
import threading
import time

BASELINE_TOK_S = 23316.0  # reference README: GPT-2 124M BF16 T=1024 on an RTX 3070 Laptop
SEQ_LEN = 1024
SEQS_PER_GPU = 16


class ClockSampler:
    """Samples SM clocks and throttle reasons while the timed region runs: NVML reads from a thread every
    20 ms (reading only; no setting is changed), nvidia-smi polling as the fallback."""

    Q = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
         "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_index: int):
        self.idx = gpu_index
        self.proc = None
        self.path = None
        self.thread = None
        self._stop = False
        self.sm, self.mx, self.reasons = [], [], set()

    def _nvml_loop(self, nv, handle):
        bits = {"hw_slowdown": nv.nvmlClocksEventReasonHwSlowdown if hasattr(nv, "nvmlClocksEventReasonHwSlowdown")
                else nv.nvmlClocksThrottleReasonHwSlowdown,
                "hw_thermal_slowdown": getattr(nv, "nvmlClocksEventReasonHwThermalSlowdown",
                                               getattr(nv, "nvmlClocksThrottleReasonHwThermalSlowdown", 0x40)),
                "sw_thermal_slowdown": getattr(nv, "nvmlClocksEventReasonSwThermalSlowdown",
                                               getattr(nv, "nvmlClocksThrottleReasonSwThermalSlowdown", 0x20)),
                "sw_power_cap": getattr(nv, "nvmlClocksEventReasonSwPowerCap",
                                        getattr(nv, "nvmlClocksThrottleReasonSwPowerCap", 0x4))}
        mx = float(nv.nvmlDeviceGetMaxClockInfo(handle, nv.NVML_CLOCK_SM))
        while not self._stop:
            try:
                self.sm.append(float(nv.nvmlDeviceGetClockInfo(handle, nv.NVML_CLOCK_SM)))
                self.mx.append(mx)
                try:
                    mask = nv.nvmlDeviceGetCurrentClocksEventReasons(handle)
                except Exception:
                    mask = nv.nvmlDeviceGetCurrentClocksThrottleReasons(handle)
                for name, bit in bits.items():
                    if mask & bit:
                        self.reasons.add(name)
            except Exception:
                pass
            time.sleep(0.02)

    def start(self):
        try:
            import pynvml as nv
            nv.nvmlInit()
            vis = os.environ.get("CUDA_VISIBLE_DEVICES")
            phys = int(vis.split(",")[self.idx]) if vis and vis.split(",")[self.idx].isdigit() else self.idx
            handle = nv.nvmlDeviceGetHandleByIndex(phys)
            self.thread = threading.Thread(target=self._nvml_loop, args=(nv, handle), daemon=True)
            self.thread.start()
            return
        except Exception:
            self.thread = None
        try:
            f = tempfile.NamedTemporaryFile("w", suffix=".csv", delete=False)
            self.path = f.name
            self.proc = subprocess.Popen(["nvidia-smi", "-i", str(self.idx), f"--query-gpu={self.Q}",
                                          "--format=csv,noheader,nounits", "-lms", "100"], stdout=f,
                                         stderr=subprocess.DEVNULL)
        except Exception:
            self.proc = None

    def stop(self) -> dict:
        out = {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        if self.thread is not None:
            self._stop = True
            self.thread.join(timeout=2)
        elif self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except Exception:
                self.proc.kill()
            try:
                for line in open(self.path):
                    p = [x.strip() for x in line.split(",")]
                    if len(p) < 9:
                        continue
                    try:
                        self.sm.append(float(p[1]))
                        self.mx.append(float(p[2]))
                    except ValueError:
                        continue
                    for name, val in zip(("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"),
                                         p[5:9]):
                        if val.lower().startswith("active"):
                            self.reasons.add(name)
                os.unlink(self.path)
            except Exception:
                pass
        if self.sm:
            out.update(sm_mhz=statistics.median(self.sm), sm_max_mhz=max(self.mx), reasons=sorted(self.reasons),
                       samples=len(self.sm))
        return out


def run_reference(args) -> int:
    """The unmodified reference on the same metric and config: its `cuda::GptModel` + `cuda::GptTrainer`
    (cuBLASLt GEMMs, its own FlashAttention-2, fused CE and foreach AdamW kernels) compiled from its sources by
    `baseline/build_ref.py` into `baseline/_ref/lib/libnexus_ref_gpt.so`.  Nothing of nexus_b200 is imported on
    this path.  The reference has no multi-GPU training path that builds offline (its GPU data-parallel backend
    sits behind `LanguageModelTrainer`, whose sources include the empty `NexusOptim` / `NexusData` submodules), so
    N > 1 reports `unavailable`."""
    import ctypes

    def unavailable(why: str) -> int:
        print(json.dumps({"impl": "reference", "unavailable": why}))
        return 0

    world = int(os.environ.get("WORLD_SIZE", "1"))
    if args.gpus > 1 or world > 1:
        if int(os.environ.get("RANK", "0")) == 0:
            return unavailable("the reference's only multi-GPU training path (cuda::gpt_backend data parallel inside "
                               "LanguageModelTrainer) does not compile offline: src/train/lm_trainer.cpp includes "
                               "headers of the empty NexusOptim / NexusData submodules; single-GPU arm only")
        return 0
    here = os.path.dirname(os.path.abspath(__file__))
    lib_path = os.path.join(here, "baseline", "_ref", "lib", "libnexus_ref_gpt.so")
    if not os.path.exists(lib_path):
        try:
            sys.path.insert(0, os.path.join(here, "baseline"))
            import build_ref
            build_ref.build(verbose=False)
        except Exception as e:  # no reference sources or no compiler on this machine
            return unavailable(("reference library not built and cannot be built here: %s" % e).splitlines()[0][:300])
    try:
        lib = ctypes.CDLL(lib_path)
    except OSError as e:
        return unavailable(("cannot load %s: %s" % (lib_path, e))[:300])
    lib.nexus_ref_gpt_error.restype = ctypes.c_char_p
    rc = lib.nexus_ref_gpt_open(args.seqs, args.seq_len, 1, 0)
    if rc != 0:
        return unavailable("reference GptModel construction failed (rc %d): %s" % (rc, lib.nexus_ref_gpt_error().decode()))
    warm = max(args.warmup, 3)
    ms, loss = ctypes.c_double(0.0), ctypes.c_float(0.0)
    sampler = ClockSampler(int(os.environ.get("LOCAL_RANK", "0")))
    sampler.start()
    rc = lib.nexus_ref_gpt_device(args.steps, warm, ctypes.byref(ms), ctypes.byref(loss))
    clocks = sampler.stop()
    if rc != 0:
        return unavailable("reference device-timed run failed (rc %d): %s" % (rc, lib.nexus_ref_gpt_error().decode()))
    e2e = None
    if not args.skip_e2e:
        ems, eloss = ctypes.c_double(0.0), ctypes.c_float(0.0)
        rc = lib.nexus_ref_gpt_e2e(args.steps, warm, ctypes.byref(ems), ctypes.byref(eloss))
        if rc == 0:
            e2e = {"value": args.seqs * args.seq_len / (ems.value * 1e-3), "unit": "tokens/s",
                   "h2d_bytes_per_step": args.seqs * args.seq_len * 4, "d2h_bytes_per_step": 4,
                   "final_loss": eloss.value}
    buf = ctypes.create_string_buffer(2048)
    lib.nexus_ref_gpt_info(buf, 2048)
    try:
        info = json.loads(buf.value.decode())
    except Exception:
        info = {}
    lib.nexus_ref_gpt_close()
    value = args.seqs * args.seq_len / (ms.value * 1e-3)
    print(json.dumps({
        "metric": "train tokens/s GPT-2 124M bf16 (FSDP-sharded optimizer when N>1)",
        "value": value, "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": warm,
        "ms_per_step": ms.value, "higher_is_better": True, "scaling": "weak",
        "vs_baseline": value / BASELINE_TOK_S, "dtype": "bf16", "data": "synthetic uniform tokens, random-init weights",
        "impl": "reference",
        "config": {"model": args.model, "global_batch": args.seqs, "seq_len": args.seq_len, "parallelism": "single",
                   "l2": "working set per step exceeds the 126 MB L2; no explicit flush",
                   "reference_path": "cuda::GptModel::forward_backward + optimizer_step; e2e: cuda::GptTrainer::step",
                   "reference_options": "BF16 autocast, FP32 master, flash attention, no recompute, vocab padded to 64, "
                                        "fused CE cast, fast CE (its compile-mode settings)",
                   "final_loss": loss.value, **info},
        "clocks": {"sm_mhz": clocks["sm_mhz"], "sm_max_mhz": clocks["sm_max_mhz"], "reasons": clocks["reasons"]},
        "e2e": e2e,
    }))
    return 0


def run_serving(args) -> int:
    """Prefill and decode throughput of Gugedra, Makuzen, Gutivik or Lukopel models (random weights, BF16) at a few sizes, and of the other
    models of the same width and depth through the same engine.  One JSON line; `value` is the design's prefill rate at the
    middle size."""
    if args.impl != "ours" or args.gpus != 1:
        print(json.dumps({"impl": args.impl, "unavailable": f"the {args.workload} workload is this framework's own, on one GPU"}))
        return 0
    sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
    if args.workload == "gugedra":
        from nexus_b200.bench.hybrid import model_lines
    elif args.workload == "makuzen":
        from nexus_b200.bench.latent import model_lines
    elif args.workload == "lukopel":
        from nexus_b200.bench.talking import model_lines
    else:
        from nexus_b200.bench.routed import model_lines
    from nexus_b200.ops import _cuda as K
    sizes = [int(s) for s in args.sizes.split(",")]
    sampler = ClockSampler(0)
    sampler.start()
    rows = model_lines(sizes, max(3, args.steps))
    clocks = sampler.stop()
    mid = rows[len(rows) // 2]
    print(json.dumps({
        "metric": f"serving tokens/s, prefill of 8 x 1024 tokens, {args.workload.capitalize()}",
        "value": mid[args.workload]["prefill_tok_s"], "unit": "tokens/s",
        "n_gpus": 1, "steps": max(3, args.steps), "warmup": 3, "higher_is_better": True, "dtype": "bf16", "impl": "ours",
        "data": "random tokens, random-init weights",
        "config": {"model": f"{args.workload}-{mid['width']}", "prefill": "8 x 1024 and 1 x 4096 tokens",
                   "decode": "64 sequences, 1024 behind", "l2": "weights exceed the 126 MB L2; no explicit flush"},
        "sizes": rows, "clocks": {"sm_mhz": clocks["sm_mhz"], "sm_max_mhz": clocks["sm_max_mhz"], "reasons": clocks["reasons"]},
        "gpu_launches": K.launch_count}))
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=20)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--model", default="gpt2-124m")
    ap.add_argument("--seqs", type=int, default=SEQS_PER_GPU)
    ap.add_argument("--seq-len", type=int, default=SEQ_LEN)
    ap.add_argument("--graph", type=int, default=-1,
                    help="trainer API replays the whole step as one CUDA graph (default: on for 1 GPU, off otherwise)")
    ap.add_argument("--skip-e2e", action="store_true")
    ap.add_argument("--workload", default="train", choices=["train", "gugedra", "makuzen", "gutivik", "lukopel"],
                    help="gugedra, makuzen, gutivik, lukopel: serving speed of that design beside the other models of equal width and depth, one GPU")
    ap.add_argument("--sizes", default="1024,2048,4096", help="widths of the serving workloads")
    args = ap.parse_args()
    if args.workload != "train":
        return run_serving(args)
    if args.impl == "reference":
        return run_reference(args)
    if args.graph < 0:
        args.graph = 1 if args.gpus == 1 else 0

    import numpy as np
    import torch

    sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
    from nexus_b200.lm.config import preset
    from nexus_b200.ops import _cuda as K
    from nexus_b200.train.lm_trainer import AdamW, LanguageTrainerBuilder, SyntheticTokens

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if world != args.gpus:
        if world == 1 and args.gpus > 1:
            raise SystemExit("launch N>1 with: python -m torch.distributed.run --nproc-per-node N bench.py --gpus N")
    torch.cuda.set_device(local_rank)
    pg = None
    if world > 1:
        from nexus_b200.parallel.process_group import init_process_group
        pg = init_process_group(backend="nccl", device=f"cuda:{local_rank}")

    cfg = preset(args.model)
    B, T = args.seqs, args.seq_len
    builder = (LanguageTrainerBuilder(cfg)
               .data(SyntheticTokens(cfg.vocab_size, seed=1234, rank=rank, world=world))
               .optimizer(AdamW(lr=6e-4, beta1=0.9, beta2=0.95, eps=1e-8, weight_decay=0.1))
               .micro_batch(B).seq_len(T).global_batch_tokens(B * T * world).grad_clip(1.0)
               .precision("bf16", "fp32").execution_policy(f"cuda:{local_rank}").log_every(0)
               .compile(bool(args.graph)))
    if pg is not None:
        builder = builder.fsdp(pg, None) if os.environ.get("NEXUS_BENCH_DDP", "0") != "1" else builder.process_group(pg)
    trainer = builder.build()
    backend = trainer.backend

    def barrier():
        if pg is not None:
            pg.barrier()
        torch.cuda.synchronize()

    # ---------------- warm-up through the public API (also builds every lazily created buffer)
    trainer.train(max(args.warmup, 3))

    # ---------------- device-timed region: K optimizer steps, inputs resident on the device
    tokens_dev = [torch.randint(0, cfg.vocab_size, (B, T), dtype=torch.int32, device=f"cuda:{local_rank}",
                                generator=torch.Generator(device=f"cuda:{local_rank}").manual_seed(100 + rank + 17 * i))
                  for i in range(4)]
    sampler = ClockSampler(local_rank)
    launches0 = K.launch_count
    barrier()
    sampler.start()
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    ev0.record()
    for i in range(args.steps):
        backend.device_step(tokens_dev[i % 4], lr=6e-4)
    ev1.record()
    barrier()
    clocks = sampler.stop()
    launches = K.launch_count - launches0
    ms = ev0.elapsed_time(ev1) / args.steps
    if pg is not None:
        ms = float(pg.all_reduce_scalar(ms, "max"))
    K.check_status()
    value = B * T * world / (ms * 1e-3)

    # ---------------- end-to-end through the public trainer API (H2D of tokens + D2H of the loss per step)
    e2e = None
    if not args.skip_e2e:
        h0, d0 = backend.h2d_bytes, backend.d2h_bytes
        barrier()
        t0 = time.perf_counter()
        trainer.train(args.steps)
        barrier()
        dt = time.perf_counter() - t0
        if pg is not None:
            dt = float(pg.all_reduce_scalar(dt, "max"))
        e2e = {"value": B * T * world * args.steps / dt, "unit": "tokens/s",
               "h2d_bytes_per_step": (backend.h2d_bytes - h0) // args.steps,
               "d2h_bytes_per_step": (backend.d2h_bytes - d0) // args.steps,
               "final_loss": trainer.history[-1].loss}

    if rank == 0:
        print(json.dumps({
            "metric": "train tokens/s GPT-2 124M bf16 (FSDP-sharded optimizer when N>1)",
            "value": value, "unit": "tokens/s", "n_gpus": world, "steps": args.steps, "warmup": max(args.warmup, 3),
            "ms_per_step": ms, "higher_is_better": True, "scaling": "weak",
            "vs_baseline": value / BASELINE_TOK_S, "dtype": "bf16", "data": "synthetic uniform tokens, random-init weights",
            "impl": "ours",
            "config": {"model": args.model, "global_batch": B * world, "seq_len": T,
                       "parallelism": f"fsdp{world}" if world > 1 else "single",
                       "l2": "working set per step (activations 7 GB) exceeds the 126 MB L2; no explicit flush",
                       "cuda_graph": bool(args.graph)},
            "clocks": {"sm_mhz": clocks["sm_mhz"], "sm_max_mhz": clocks["sm_max_mhz"], "reasons": clocks["reasons"]},
            "e2e": e2e, "gpu_launches": launches,
        }))
    if pg is not None:
        pg.destroy()
    return 0


if __name__ == "__main__":
    sys.exit(main())
