#!/usr/bin/env python
"""Headline benchmark: Llama-3-8B-shaped full fine-tune, FSDP2 bf16, seq 8192, micro-batch 1 per GPU,
synthetic uniform-random tokens, random-init weights.  Prints ONE JSON line on rank 0.

  python bench.py --gpus 1 --steps 5 --warmup 3
  python -m torch.distributed.run --nnodes=1 --nproc-per-node 8 --master-addr 127.0.0.1 --master-port 29511 \
      bench.py --gpus 8 --steps 5 --warmup 3
  python bench.py --impl reference ...      # the unmodified reference from baseline/_ref, same metric/config

`value` is device-timed (CUDA events, barrier + synchronize on both sides, max over ranks) with batches that
already sit on the device; `e2e` times the same steps through `SOTATrainer.train_step`, which copies each batch
from pinned host memory and reads the loss back every step.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

MODEL = "llama3-8b"
SEQ = 8192
MICRO_BATCH = 1


class ClockSampler:
    """Samples SM clock / throttle reasons with nvidia-smi while the timed region runs."""
    Q = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
         "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
         "clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.index, self.samples, self.proc = index, [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--id={self.index}", f"--query-gpu={self.Q}",
                                          "--format=csv,noheader,nounits", "-lms", "200"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.samples.append([x.strip() for x in line.split(",")])

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
        for s in self.samples:
            try:
                sm.append(float(s[0]))
                mx = float(s[1])
            except (ValueError, IndexError):
                continue
            for n, v in zip(names, s[3:7]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": mx, "reasons": sorted(reasons),
                "samples": len(sm)}


def baseline_value(n_gpus: int = 1) -> float | None:
    """The number `vs_baseline` divides by: a published value from BASELINE.json when the reference publishes one (it
    does not), else the reference's own throughput measured on this pool's B200s at the same GPU count
    (baseline/measured_reference.json)."""
    try:
        pub = json.loads((ROOT / "BASELINE.json").read_text()).get("published", {})
        for v in pub.values():
            if isinstance(v, (int, float)):
                return float(v)
    except Exception:
        pass
    try:
        ref = json.loads((ROOT / "baseline" / "measured_reference.json").read_text())["tokens_per_s"]
        v = ref.get(str(n_gpus))
        return float(v) if v else None
    except Exception:
        return None


def run_ours(args) -> dict:
    """Headline measurement with `--sharding`, then (2+ GPUs) a shorter one with the other ZeRO mode whose value is
    reported inside `config` (`other_sharding`).  The process group is created once here so that both trainers share
    it.  A watchdog prints the headline line alone if the second measurement does not finish."""
    import gc

    import torch
    import torch.distributed as dist

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    torch.cuda.set_device(local)
    if world > 1 and not dist.is_initialized():
        dist.init_process_group("nccl", rank=rank, world_size=world, device_id=torch.device("cuda", local))
    out = measure(args, args.sharding, args.steps, args.warmup)
    other = {"full_shard": "shard_grad_op", "full": "shard_grad_op"}.get(args.sharding, "full_shard")
    if world > 1 and not args.no_secondary:
        line = json.dumps(out)

        def give_up():
            if rank == 0:
                print(line, flush=True)
            os._exit(0)

        dog = threading.Timer(args.secondary_timeout, give_up)
        dog.daemon = True
        dog.start()
        try:
            gc.collect()
            torch.cuda.empty_cache()
            torch.cuda.reset_peak_memory_stats()
            sec = measure(args, other, min(args.steps, 6), 3, e2e=False)
            if rank == 0:
                out["config"]["other_sharding"] = {"sharding": other, "value": sec["value"], "unit": "tokens/s",
                                                   "ms_per_step": sec["ms_per_step"], "steps": sec["steps"],
                                                   "peak_mem_gb": sec["peak_mem_gb"]}
        except Exception as e:   # noqa: BLE001 - the headline stands on its own
            if rank == 0:
                out["config"]["other_sharding"] = {"sharding": other, "error": f"{type(e).__name__}: {e}"[:200]}
        dog.cancel()
    if world > 1:
        dist.barrier()
        dist.destroy_process_group()
    return out


def measure(args, sharding: str, steps: int, warmup: int, e2e: bool = True) -> dict:
    import torch
    import torch.distributed as dist

    from trainscale_b200.config.sota_config import SOTAConfig
    from trainscale_b200.models.llama import preset_config
    from trainscale_b200.ops import _lib
    from trainscale_b200.trainer.sota_trainer import SOTATrainer

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    torch.cuda.set_device(local)
    mcfg = preset_config(args.model)
    seq, mb = args.seq, args.micro_batch
    # one GPU holds all 128 GB of parameter/optimizer state: keep only the GEMM-side activations there
    ac = args.ac if args.ac != "auto" else ("op_selective" if world == 1 else "none")
    layer_ckpt = ac in ("full", "half")
    cfg = SOTAConfig.from_dict({
        "training_mode": "full",
        "model": {"architecture": args.model},
        "optimizer": {"type": "adamw", "learning_rate": 2e-5, "weight_decay": 0.01, "max_grad_norm": 1.0},
        "scheduler": {"type": "cosine", "warmup_steps": 2},
        "loss": {"type": "chunked_ce"},
        "distributed": {"enabled": world > 1, "backend": "nccl", "strategy": "fsdp2", "world_size": world,
                        "gradient_checkpointing": layer_ckpt, "comm": args.comm,
                        "fsdp_config": {"sharding_strategy": sharding, "activation_checkpointing": layer_ckpt,
                                        "ac_mode": ac, "ac_frequency": 2 if ac == "half" else 1,
                                        "gradient_accumulation_steps": 1}},
        "hardware": {"precision": "bf16"},
        "data": {"max_seq_length": seq},
        "training": {"per_device_train_batch_size": mb, "gradient_accumulation_steps": 1, "max_steps": 10 ** 6,
                     "logging_steps": 10 ** 9, "save_strategy": "no", "save_steps": 0, "eval_strategy": "no",
                     "early_stopping_patience": 0, "output_dir": "/tmp/ts_bench_out"},
    })
    trainer = SOTATrainer(cfg)
    trainer.setup_model()
    trainer.setup_optimizer()
    trainer.setup_scheduler(10 ** 6)
    dev = trainer.device
    n_batches = warmup + steps
    g = torch.Generator().manual_seed(1234 + rank)
    host = [torch.randint(0, mcfg.vocab_size, (mb, seq), generator=g, dtype=torch.int64).pin_memory()
            for _ in range(n_batches)]
    devb = [h.to(dev) for h in host]

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    def device_step(ids):
        loss, _ = trainer._forward_loss({"input_ids": ids, "labels": ids}, 1.0)
        trainer.engine.micro_step = 0
        trainer.engine.backward(loss)
        trainer.engine.step(trainer.optimizer.param_groups[0]["lr"])
        trainer.scheduler.step()
        return loss

    # ---- device-timed region
    for i in range(warmup):
        try:
            device_step(devb[i])
        except torch.OutOfMemoryError:
            # the automatic one-GPU policy did not fit beside this process's other allocations: recompute every
            # second layer instead (the warm-up restarts, so the timed steps see one policy only)
            if not (args.ac == "auto" and ac == "op_selective" and i == 0):
                raise
            ac = "half"
            trainer.model.op_selective_recompute(False)
            trainer.model.gradient_checkpointing_enable(2)
            trainer.engine.zero_grad()
            torch.cuda.empty_cache()
            device_step(devb[i])
    barrier()
    sampler = ClockSampler(local)
    if rank == 0:
        sampler.start()
    launches0 = _lib.LAUNCHES
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for i in range(steps):
        loss = device_step(devb[warmup + i])
    e1.record()
    barrier()
    launches = _lib.LAUNCHES - launches0
    ms = e0.elapsed_time(e1)
    final_loss = float(loss.detach())
    # ---- end-to-end region through the public API (H2D from pinned memory + loss read each step)
    ms_e2e = ms
    if e2e:
        for i in range(min(2, warmup)):
            trainer.train_step({"input_ids": host[i], "labels": host[i]})
        barrier()
        f0, f1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        f0.record()
        for i in range(steps):
            h = host[warmup + i]
            trainer.train_step({"input_ids": h, "labels": h})
        f1.record()
        barrier()
        ms_e2e = f0.elapsed_time(f1)
    clocks = sampler.stop() if rank == 0 else None
    t = torch.tensor([ms, ms_e2e], device=dev)
    if world > 1:
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
    ms, ms_e2e = (float(x) for x in t.tolist())
    _lib.raise_on_any_device_error()
    tokens_per_step = mb * seq * world
    value = tokens_per_step * steps / (ms / 1e3)
    e2e_value = tokens_per_step * steps / (ms_e2e / 1e3)
    peaks = {}
    try:
        peaks = json.loads((ROOT / "MEASURED_PEAKS.json").read_text())
    except Exception:
        pass
    flops_tok = mcfg.flops_per_token(seq)
    peak = float(peaks.get("bf16_tflops_sustained", 1385.7))
    base = baseline_value(world)
    out = {
        "metric": "train tokens/s/box (Llama-3-8B FSDP2 bf16)", "value": value, "unit": "tokens/s", "n_gpus": world,
        "steps": steps, "warmup": warmup, "ms_per_step": ms / steps, "higher_is_better": True,
        "scaling": "weak", "vs_baseline": (value / base) if base else None, "dtype": "bf16",
        "data": "synthetic uniform-random tokens, random-init weights", "impl": "ours",
        "config": {"model": args.model, "global_batch": mb * world, "seq_len": seq,
                   "parallelism": f"fsdp{world}" if world > 1 else "single", "sharding": sharding,
                   "activation_checkpointing": ac, "comm": args.comm,
                   "l2": "inputs (16 GB of weights per step) are larger than L2; no explicit flush"},
        "mfu_of_measured_sustained_peak": value * flops_tok / 1e12 / (peak * world),
        "clocks": clocks,
        "e2e": {"value": e2e_value, "unit": "tokens/s", "ms_per_step": ms_e2e / steps,
                "h2d_bytes_per_step": int(host[0].numel() * host[0].element_size()) * world,
                "d2h_bytes_per_step": 4 * world},
        "gpu_launches": launches, "final_loss": final_loss,
        # torch's allocator peak plus the symmetric-memory buffers (flat parameters / gradients of the fused path),
        # which are allocated outside it
        "peak_mem_gb": (torch.cuda.max_memory_allocated() +
                        getattr(getattr(trainer.engine, "_symm", None), "bytes_allocated", 0)) / 2 ** 30,
    }
    trainer.cleanup()
    del trainer, devb
    return out if rank == 0 else {"value": value, "ms_per_step": ms / steps, "steps": steps, "peak_mem_gb": 0.0,
                                  "config": {}}


def run_serving(args) -> None:
    """One JSON line per size; device-timed, L2 flushed between steps, random weights and tokens."""
    from trainscale_b200.inference import bench_serving
    sampler = ClockSampler(0)
    for size in args.serve or list(bench_serving.DESIGNS[args.serve_model].sizes):
        sampler.samples.clear()
        sampler.start()
        res = bench_serving.run([size], ROOT / "MEASURED_PEAKS.json", max(args.steps, 5),
                                args.serve_model)[size]
        print(json.dumps({"design": args.serve_model, "size": size, "dtype": "bf16", "data": "random weights and tokens", **res,
                          "clocks": sampler.stop()}), flush=True)


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=5)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--model", default=MODEL)
    ap.add_argument("--seq", type=int, default=SEQ)
    ap.add_argument("--micro-batch", type=int, default=MICRO_BATCH)
    ap.add_argument("--ac", default="auto", choices=["auto", "full", "half", "op_selective", "none"])
    ap.add_argument("--sharding", default="full_shard", choices=["full", "full_shard", "shard_grad_op", "no_shard"])
    ap.add_argument("--comm", default="auto", choices=["auto", "fused", "nccl"])
    ap.add_argument("--no-secondary", action="store_true", help="skip the measurement of the other sharding mode")
    ap.add_argument("--secondary-timeout", type=float, default=300.0)
    ap.add_argument("--serve", nargs="*", default=None, metavar="SIZE",
                    help="instead: prefill / decode throughput of a served design beside the closest model at these "
                         "sizes (default all), with per-op roofline fractions; one GPU")
    ap.add_argument("--serve-model", default="mezilix", choices=["mezilix", "vibepel", "kabulix", "lovurax"], help="design that --serve measures")
    args = ap.parse_args()
    if args.serve is not None:
        return run_serving(args)
    args.warmup = max(args.warmup, 3)
    world = int(os.environ.get("WORLD_SIZE", "1"))
    if args.gpus > 1 and world == 1:
        # convenience: relaunch under torchrun
        cmd = [sys.executable, "-m", "torch.distributed.run", "--nnodes=1", f"--nproc-per-node={args.gpus}",
               "--master-addr", "127.0.0.1", "--master-port", os.environ.get("MASTER_PORT", "29533"),
               str(Path(__file__).resolve())] + sys.argv[1:]
        raise SystemExit(subprocess.call(cmd))
    if args.impl == "reference":
        from baseline.reference_runner import run_reference
        out = run_reference(args)
    else:
        out = run_ours(args)
    if out and int(os.environ.get("RANK", "0")) == 0:
        print(json.dumps(out), flush=True)


if __name__ == "__main__":
    main()
