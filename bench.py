#!/usr/bin/env python
"""Headline benchmark: training throughput (tokens/s over the whole job) of the dense 1.3B
OIL8-STE model — 24 layers, d 2048, 16 heads, SwiGLU 5504, vocab 32000, seq 2048 — with bf16
compute, fp32 master weights, STE fake-quantised linear weights, fused AdamW, ZeRO-style data
parallel. Weak scaling: 64 sequences per GPU per optimizer step (global batch 512 at 8 GPUs).
Synthetic seeded Zipf(1.1) tokens, random-init N(0, 0.02) weights.

    python bench.py --gpus 1 --steps 5 --warmup 3
    python -m torch.distributed.run --nnodes=1 --nproc-per-node 8 --master-addr 127.0.0.1 \
        --master-port 29500 bench.py --gpus 8 --steps 5 --warmup 3

After the training measurement the same process group runs the second half of the headline metric:
greedy decode of a Llama-3-8B-shaped model (mixed OIL4 attention / OIL8 FFN weights, paged bf16 KV
with 16-token pages, batch 64, prompt 1024, 256 new tokens) with tensor parallelism over the N
GPUs of the run; tokens/s, p50 time to first token and the fraction of the HBM bound are reported in
the ``decode`` object of the same JSON line (``--no-decode`` skips it).

Prints one JSON line on rank 0. ``--impl reference`` reports why the reference cannot run this
configuration (CPU-only FP32 C++ engine without a Python package, a GPU path or multi-process
communication).
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

SEQ = 2048
PER_GPU_BATCH = 64
MICRO_BATCH = 32     # sequences per forward/backward pass; measured 104.0k / 110.5k / 112.4k tokens/s at 8 / 16 / 32 (peak 124 GB at 32)


class ClockSampler:
    """Samples SM clocks and throttle reasons of one GPU with nvidia-smi while the timed region runs."""

    FIELDS = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
              "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
              "clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int):
        self.index = index
        self.proc = None
        self.lines: list[str] = []
        self.thread = None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--id={self.index}", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits",
                 "-lms", "200"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.proc = None
            return
        self.thread = threading.Thread(target=self._pump, daemon=True)
        self.thread.start()

    def _pump(self):
        for line in self.proc.stdout:
            self.lines.append(line.strip())

    def stop(self) -> dict:
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for ln in self.lines:
            parts = [p.strip() for p in ln.split(",")]
            if len(parts) < 7:
                continue
            try:
                sm.append(float(parts[0]))
                mx.append(float(parts[1]))
            except ValueError:
                continue
            for n, v in zip(names, parts[3:7]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        # the busiest half of the samples is "under load"
        sm_sorted = sorted(sm)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "sm_mhz_min": sm_sorted[0] if sm else None, "samples": len(sm), "reasons": sorted(reasons)}


def model_flops_per_token(cfg) -> float:
    d, L, f, V, S = cfg.hidden_size, cfg.num_layers, cfg.ffn_hidden_size, cfg.vocab_size, SEQ
    lin = L * (d * (cfg.q_dim + 2 * cfg.kv_dim) + cfg.q_dim * d + 3 * d * f) + V * d
    attn = L * 2 * S * cfg.q_dim * 0.5 * 2  # QK^T and PV, causal half
    return 6.0 * lin + 3.0 * attn


def run_decode(world: int, rank: int, device, args, hbm_gbs: float) -> dict:
    """TP = world decode benchmark of the Llama-3-8B-shaped mixed OIL4 / OIL8 model (the second half
    of the headline metric). Device-side decode time, max over ranks; TTFT is prefill + first sample
    around a device synchronise, p50 over the timed repeats, max over ranks."""
    import torch

    from mythos_b200.infer.engine import InferenceEngine, TPContext
    from mythos_b200.models.config import NAMED_CONFIGS
    from mythos_b200.ops import native

    cfg = NAMED_CONFIGS["llama3-8b"]()
    batch, prompt, new = args.decode_batch, args.decode_prompt, args.decode_new
    cfg.max_seq_len = prompt + new + 16
    tp = None
    if world > 1:
        import torch.distributed as dist

        tp = TPContext(dist.group.WORLD, device, max_tokens=max(batch * prompt, 256), hidden=cfg.hidden_size,
                       vocab_shard=cfg.vocab_size // world, max_batch=batch)
    torch.manual_seed(1234)
    eng = InferenceEngine.random(cfg, seed=1234, device=device, max_batch=batch, max_seq_len=cfg.max_seq_len, tp=tp,
                                 kv_dtype="bf16")
    wbytes = eng.weight_bytes()
    torch.cuda.empty_cache()
    g = torch.Generator().manual_seed(7)
    prompts = torch.randint(0, cfg.vocab_size, (batch, prompt), generator=g, dtype=torch.int32)
    ttfts, dec_s = [], []
    launches0 = native.launch_count()
    for it in range(args.decode_repeat + 1):                       # the first repeat is the warm-up
        res = eng.generate(prompts, max_new_tokens=new, use_graph=True)
        t = torch.tensor([res.stats.ttft_s, res.stats.decode_s], device=device, dtype=torch.float64)
        if world > 1:
            import torch.distributed as dist

            dist.all_reduce(t, op=dist.ReduceOp.MAX)
        if it > 0:
            ttfts.append(float(t[0]))
            dec_s.append(float(t[1]))
    native.check_status(device)
    ttfts.sort()
    best = min(dec_s)
    ms_step = best / (new - 1) * 1e3
    # bytes one rank must stream per decode step: its weight shard once, its share of the KV pages
    # at the mean context length of the decode phase
    kv_per_tok = 2 * cfg.num_layers * (cfg.kv_dim // world if world <= cfg.kv_heads else cfg.head_dim) * 2
    kv_bytes = batch * (prompt + new / 2) * kv_per_tok
    bound_ms = (wbytes + kv_bytes) / (hbm_gbs * 1e9) * 1e3
    return {"metric": "TP decode tok/s, p50 TTFT", "tp": world, "tok_s": batch * (new - 1) / best,
            "p50_ttft_s": ttfts[len(ttfts) // 2], "ms_per_step": ms_step,
            "config": {"model": "llama3-8b shape (32L d4096 32q/8kv ffn14336 v128256), OIL4 attention / OIL8 FFN + embeddings",
                       "batch": batch, "prompt": prompt, "new_tokens": new, "kv": "paged bf16, 16-token pages",
                       "sampling": "greedy", "decode": "CUDA-graph replay"},
            "weight_bytes_per_rank": int(wbytes), "kv_bytes_read_per_step_per_rank": int(kv_bytes),
            "hbm_bound_ms_per_step": bound_ms, "fraction_of_hbm_bound": bound_ms / ms_step,
            "decode_s_runs": [round(x, 4) for x in dec_s],
            "gpu_launches": int(native.launch_count() - launches0),
            "data": "random-init weights in format, uniform-random prompts"}


def run_reference_arm():
    print(json.dumps({"impl": "reference", "unavailable":
                      "reference is a CPU-only FP32 C++ engine (no setup.py/pyproject: pip install fails; no GPU "
                      "path, no bf16, no multi-process data parallel), so the 1.3B bf16 ZeRO config cannot run on it"}))
    return 0


def run_hybrid(design: str) -> int:
    """Layer-list models beside the dense engine (mythos_b200/tools/hybrid_bench.py)."""
    from mythos_b200.tools import hybrid_bench

    peaks = {}
    try:
        with open(os.path.join(os.path.dirname(os.path.abspath(__file__)), "MEASURED_PEAKS.json")) as f:
            peaks = json.load(f)
    except OSError:
        pass
    sampler = ClockSampler(0)
    sampler.start()
    models, kernels = hybrid_bench.run_models(design), hybrid_bench.run_kernels(peaks, design=design)
    print(json.dumps({"metric": "hybrid prefill / decode throughput", "n_gpus": 1, "dtype": "bf16", "models": models,
                      "kernels": kernels, "clocks": sampler.stop(), "data": "random-init weights, uniform-random prompts"}))
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=4)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--per-gpu-batch", type=int, default=PER_GPU_BATCH)
    ap.add_argument("--micro-batch", type=int, default=MICRO_BATCH)
    ap.add_argument("--dp-mode", default="fused", choices=["fused", "nccl"],
                    help="data-parallel gradient path: fused peer-memory kernels or plain NCCL collectives")
    ap.add_argument("--activation-checkpointing", action="store_true",
                    help="recompute block activations in the backward pass (memory for one extra forward)")
    ap.add_argument("--hybrid", nargs="?", const="teganex", default=None, choices=["teganex", "lebedra", "dogozen", "zigivik"],
                    help="instead of the headline workload: prefill / decode throughput and kernel times of layer-list layers "
                         "of this design (default: teganex) beside the dense engine of equal size, one JSON line (1 GPU)")
    ap.add_argument("--no-decode", action="store_true", help="skip the tensor-parallel decode measurement")
    ap.add_argument("--decode-batch", type=int, default=64)
    ap.add_argument("--decode-prompt", type=int, default=1024)
    ap.add_argument("--decode-new", type=int, default=256)
    ap.add_argument("--decode-repeat", type=int, default=2)
    args = ap.parse_args()
    if args.impl == "reference":
        return run_reference_arm()

    import torch

    sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
    if args.hybrid:
        return run_hybrid(args.hybrid)
    from mythos_b200.models import DenseModel
    from mythos_b200.models.config import llama_1p3b_config
    from mythos_b200.ops import native
    from mythos_b200.train.data import ZipfStream
    from mythos_b200.train.trainer import TrainConfig, Trainer

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if world != args.gpus and world > 1:
        raise SystemExit(f"--gpus {args.gpus} but WORLD_SIZE={world}")
    torch.cuda.set_device(local_rank)
    device = torch.device("cuda", local_rank)
    native.require()

    dp = None
    if world > 1:
        import torch.distributed as dist

        dist.init_process_group("nccl", device_id=device)
        from mythos_b200.parallel.zero import ZeroEngine

        dp = ZeroEngine(dist.group.WORLD, device, mode=args.dp_mode)

    cfg = llama_1p3b_config()
    torch.manual_seed(1234)
    with torch.device(device):
        model = DenseModel(cfg)
    tcfg = TrainConfig(batch_size=args.per_gpu_batch, micro_batch_size=args.micro_batch, seq_length=SEQ, lr=3e-4,
                       warmup_steps=100, max_steps=10000, max_grad_norm=1.0, codebook_ema_interval=0,
                       activation_checkpointing=args.activation_checkpointing)
    trainer = Trainer(model, tcfg, device=device, dp=dp)
    stream = ZipfStream(cfg.vocab_size, args.per_gpu_batch, SEQ, s=1.1, seed=100 + rank, pin=True)

    def barrier():
        if dp is not None:
            dp.barrier()
        torch.cuda.synchronize()

    # device-resident batches for the kernel-only measurement, pinned-host batches for end-to-end
    dev_batches = [tuple(t.to(device) for t in stream.next_batch()) for _ in range(2)]
    host_batches = [stream.next_batch() for _ in range(2)]

    for i in range(args.warmup):
        ids, tg = dev_batches[i % 2]
        trainer.train_step(ids, tg)
    barrier()
    native.check_status(device)

    sampler = ClockSampler(local_rank)
    sampler.start()
    launches0 = native.launch_count()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    barrier()
    native.require().comm_barrier_wait_stats(True)   # device-side wait counters of the flag barriers: cleared
    e0.record()
    for i in range(args.steps):
        ids, tg = dev_batches[i % 2]
        loss = trainer.train_step(ids, tg)
    e1.record()
    torch.cuda.synchronize()
    n_bar, wait_cycles, longest_cycles = native.require().comm_barrier_wait_stats(True)
    barrier()
    dev_ms = e0.elapsed_time(e1)
    launches = native.launch_count() - launches0

    # end to end through the public API: pinned host -> device each step, loss read back each step
    barrier()
    t0 = time.perf_counter()
    last = 0.0
    for i in range(args.steps):
        ids, tg = host_batches[i % 2]
        last = trainer.train_step(ids, tg).item()
    barrier()
    e2e_s = time.perf_counter() - t0
    clocks = sampler.stop()
    native.check_status(device)

    # cycles between a rank's arrival at a flag barrier and the last peer's, converted with the SM clock
    # sampled during the run: how long this rank sat waiting for the others, per step
    mhz = float(clocks.get("sm_mhz") or 0) or 1700.0
    wait_ms = wait_cycles / (mhz * 1e3) / max(1, args.steps)
    longest_ms = longest_cycles / (mhz * 1e3)
    t = torch.tensor([dev_ms, e2e_s * 1e3, wait_ms, longest_ms], device=device, dtype=torch.float64)
    tsum = torch.tensor([wait_ms], device=device, dtype=torch.float64)
    if dp is not None:
        import torch.distributed as dist

        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        dist.all_reduce(tsum, op=dist.ReduceOp.SUM)
    dev_ms, e2e_ms = float(t[0]), float(t[1])
    barrier_wait = {"barriers_per_step": n_bar / max(1, args.steps), "mean_ms_per_step": float(tsum[0]) / world,
                    "max_ms_per_step": float(t[2]), "longest_single_wait_ms": float(t[3]),
                    "note": "device cycle counters in the flag-barrier kernel (arrival -> last peer), mean / max over ranks"}
    tokens_per_step = args.per_gpu_batch * SEQ * world
    value = tokens_per_step * args.steps / (dev_ms / 1e3)
    e2e_value = tokens_per_step * args.steps / (e2e_ms / 1e3)
    peaks = {}
    try:
        with open(os.path.join(os.path.dirname(os.path.abspath(__file__)), "MEASURED_PEAKS.json")) as f:
            peaks = json.load(f)
    except OSError:
        pass
    peak_tflops = peaks.get("bf16_tflops_sustained", 1400.0)
    mfu = value / world * model_flops_per_token(cfg) / (peak_tflops * 1e12)
    peak_mem_gb = torch.cuda.max_memory_allocated(device) / 2 ** 30
    flops_per_token = model_flops_per_token(cfg)

    decode = None
    if not args.no_decode:
        # release the training state (weights, optimizer shards, activations cache) before the engine is built
        import gc

        del trainer, model, stream, dev_batches, host_batches, loss
        if dp is not None:
            dp.release()
        dp = None
        gc.collect()
        torch.cuda.empty_cache()
        try:
            decode = run_decode(world, rank, device, args, float(peaks.get("hbm_gbs", 6650.0)))
        except Exception as e:                                   # the training line must still be printed
            decode = {"error": f"{type(e).__name__}: {e}"}
    if rank == 0:
        h2d = 2 * args.per_gpu_batch * SEQ * 4
        out = {
            "metric": "train tok/s/box (1.3B OIL8-STE)", "value": value, "unit": "tokens/s", "n_gpus": world,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": dev_ms / args.steps,
            "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
            "data": "synthetic seeded Zipf(1.1) tokens, random-init N(0,0.02) weights and quantile codebooks",
            "config": {"model": "dense-1.3B (24L d2048 16h ffn5504 v32000) OIL8 STE on all linear weights",
                       "global_batch": args.per_gpu_batch * world, "seq_len": SEQ,
                       "micro_batch": args.micro_batch,
                       "activation_checkpointing": bool(args.activation_checkpointing),
                       "parallelism": f"dp{world}-zero" + (f"-{args.dp_mode}" if world > 1 else ""),
                       "l2": "working set (weights 2.6 GB + activations) far exceeds the 126 MB L2; no flush needed",
                       "optimizer": "AdamW fp32 master, global-norm clip 1.0, every step inside the timed region"},
            "clocks": clocks,
            "e2e": {"value": e2e_value, "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": 4,
                    "ms_per_step": e2e_ms / args.steps},
            "gpu_launches": int(launches),
            "barrier_wait": barrier_wait,
            "model_flops_per_token": flops_per_token,
            "fraction_of_measured_bf16_sustained": mfu,
            "final_loss": last,
            "peak_memory_gb": peak_mem_gb,
        }
        if decode is not None:
            out["decode"] = decode
        print(json.dumps(out))
    if world > 1:
        import torch.distributed as dist

        dist.destroy_process_group()
    return 0


if __name__ == "__main__":
    sys.exit(main())
