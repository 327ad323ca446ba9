#!/usr/bin/env python
"""bench.py — decode tokens/s of the B200 decode hot path (BASELINE.json metric).

    python bench.py --gpus N --steps K --warmup W             # this repo's arm
    python bench.py --impl reference --gpus N --steps K ...   # CPU arm (oracle port) on host cores
    torchrun --nnodes=1 --nproc-per-node N ... bench.py --gpus N ...   (N > 1: tensor parallel)

Workload (config.workload): Llama-3-8B shapes, AWQ int4 g=128 decoder linears + bf16 lm_head,
random-init weights, batch 64 sequences each with kv_len 2048 in a paged KV cache (block_size 8,
shuffled block ids), one decode token per sequence per step.  A "step" is one full decode step
(32 layers + final norm + lm_head + greedy argmax) = 64 tokens.

`value`   : device-timed (CUDA events) CUDA-graph replays, inputs resident in HBM.
`e2e`     : the same step driven through the public API with per-step host metadata build,
            pinned H2D copies of that metadata and a D2H read of the 64 sampled token ids;
            kv_len grows by one each step.
`roofline`: the dominant kernel (paged attention) timed alone with CUDA events, rotating over
            the 32 per-layer caches (17 GB > L2), algorithmic bytes / time vs the measured HBM peak.
`cpu_baseline` / `--impl reference`: oracle port of the same step on the host cores, bounded
            sample (a few layers + lm_head, extrapolated to 32 layers).
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
sys.path.insert(0, ROOT)

METRIC = "decode_tokens_per_s"
UNIT = "tokens/s"


def parse():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=20)
    ap.add_argument("--ttft", action="store_true", help="(default now) kept for old command lines")
    ap.add_argument("--no-ttft", action="store_true",
                    help="skip the unloaded p50 time-to-first-token measurement (chunked prefill of 8 "
                         "requests, ~1 s of GPU time)")
    ap.add_argument("--ttft-chunk", type=int, default=2048,
                    help="prefill chunk (token budget per step) of the TTFT measurement (default: the whole "
                         "prompt in one step, as an unloaded server would schedule it); chunks > 256 tokens "
                         "run the int4 linears as dequant + library bf16 GEMM unless B200_W4_PREFILL_DENSE=0")
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", default="b200", choices=["b200", "reference"])
    ap.add_argument("--batch", type=int, default=64)
    ap.add_argument("--seqlen", type=int, default=2048)
    ap.add_argument("--block-size", type=int, default=8)
    ap.add_argument("--quant", default="awq", choices=["awq", "gptq", "none"])
    ap.add_argument("--model", default="llama3-8b", choices=["llama3-8b", "llama3-70b"],
                    help="llama3-70b = SURVEY §8d config 4 (run it as --gpus 8 --batch 32 --seqlen 4096 "
                         "--quant gptq); the default is the configuration the metric is quoted on")
    ap.add_argument("--layers", type=int, default=None, help="debug only; the default is the named config")
    ap.add_argument("--no-graph", action="store_true")
    ap.add_argument("--skip-cpu-baseline", action="store_true")
    ap.add_argument("--arch", default="llama", choices=["llama", "kigalix", "pokadra", "zomurax", "fesupel", "gugalorn", "palulorn"],
                    help="kigalix / pokadra / zomurax / fesupel / gugalorn / palulorn: prefill / decode throughput of that design beside the Llama "
                         "decoder (zomurax and fesupel also beside kigalix, gugalorn beside fesupel, palulorn beside fesupel, gugalorn and pokadra) at equal size through the serving engine (scalellm_b200/arch_bench.py); the default "
                         "workload and its JSON line are untouched")
    ap.add_argument("--arch-size", default="all", choices=["all", "w2048", "w4096"])
    ap.add_argument("--arch-batch", type=int, default=16)
    ap.add_argument("--arch-seqlen", type=int, default=1024)
    return ap.parse_args()


def workload_name(a, world):
    q = {"awq": "AWQ-int4 g128", "gptq": "GPTQ-int4 g128", "none": "bf16"}[a.quant]
    name = {"llama3-8b": "Llama-3-8B", "llama3-70b": "Llama-3-70B"}[a.model]
    return (f"{name} {q} decode step, batch {a.batch}, kv_len {a.seqlen}, block_size "
            f"{a.block_size}, TP={world}")


# --------------------------------------------------------------------------------------
# clocks sampling (B200_PROFILING.md recipe)
# --------------------------------------------------------------------------------------
class ClockSampler:
    Q = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
         "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
         "clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int):
        self.rows, self.proc = [], None
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--id={index}", f"--query-gpu={self.Q}",
                 "--format=csv,noheader,nounits", "-lms", "100"], stdout=subprocess.PIPE,
                stderr=subprocess.DEVNULL, text=True)
            self.t = threading.Thread(target=self._read, daemon=True)
            self.t.start()
        except Exception:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append((time.perf_counter(), line.strip()))

    def window(self, t0, t1):
        return [r for (t, r) in self.rows if t0 <= t <= t1] or [r for (_, r) in self.rows[-3:]]

    def stop(self):
        if self.proc:
            self.proc.terminate()

    @staticmethod
    def summarise(rows):
        sm, mx, reasons = [], 0, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for r in rows:
            f = [x.strip() for x in r.split(",")]
            if len(f) < 7:
                continue
            try:
                sm.append(float(f[0]))
                mx = max(mx, float(f[1]))
            except ValueError:
                continue
            for n, v in zip(names, f[3:7]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        sm.sort()
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": mx or None,
                "reasons": sorted(reasons), "samples": len(sm)}


# --------------------------------------------------------------------------------------
# CPU arm: oracle port of the same decode step on the host cores
# --------------------------------------------------------------------------------------
class CpuDecodeSample:
    """Oracle port of the decode step at the benchmark shapes (built once, timed many times)."""

    SAMPLE_BATCH = 8   # sequences of the batch the CPU sample runs (same kv_len, same shapes)

    def __init__(self, a, seed: int = 0):
        import numpy as np
        import torch
        from oracle import llama as ollama, ops, quant

        torch.set_num_threads(os.cpu_count() or 1)
        self.torch, self.ollama, self.ops, self.quant = torch, ollama, ops, quant
        cfg = self.cfg = ollama.LlamaConfig()
        B, S, bs = min(a.batch, self.SAMPLE_BATCH), a.seqlen, a.block_size
        self.B = B
        g = torch.Generator().manual_seed(seed)
        h, D, H, Hkv, I = cfg.hidden, cfg.head_dim, cfg.n_heads, cfg.n_kv_heads, cfg.inter

        def lin(K, N):  # dequantised int4 weight (the CPU path multiplies dense bf16 weights)
            q = torch.randint(0, 16, (K, N), generator=g, dtype=torch.int32).numpy()
            z = torch.randint(0, 16, (K // 128, N), generator=g, dtype=torch.int32).numpy()
            s = (torch.randn(K // 128, N, generator=g).abs() * 0.01 + 1e-4).bfloat16()
            return ollama.Linear(quant.dequant(q, z, s, 128))

        self.layer = dict(qkv=lin(h, (H + 2 * Hkv) * D), o=lin(H * D, h), gate_up=lin(h, 2 * I),
                          down=lin(I, h), input_norm=torch.ones(h).bfloat16(),
                          post_norm=torch.ones(h).bfloat16())
        nblk = (S + bs - 1) // bs
        n_slots = B * nblk * bs
        self.kc = torch.randn(n_slots, Hkv, D, generator=g).bfloat16()
        self.vc = torch.randn(n_slots, Hkv, D, generator=g).bfloat16()
        table = (torch.randperm(B * nblk, generator=g) * bs).to(torch.int32)
        self.meta = dict(q_cu_lens=np.arange(B + 1), kv_cu_lens=np.arange(B + 1) * S,
                         block_table=table, block_cu_lens=np.arange(B + 1) * nblk, block_size=bs)
        last = torch.arange(B) * nblk + (S - 1) // bs
        self.slots = (table[last] + (S - 1) % bs).to(torch.int32)
        self.cos_sin = ops.build_cos_sin_cache(D, 4096, ollama.inv_freq_for(cfg), torch.bfloat16)
        self.x = (torch.randn(B, h, generator=g) * 0.5).bfloat16()
        self.pos = torch.full((B,), S - 1, dtype=torch.int32)
        self.lm_head = ollama.Linear((torch.randn(h, cfg.vocab, generator=g) * 0.02).bfloat16())
        self.fn = torch.ones(h).bfloat16()
        self._pick_threads()

    def _pick_threads(self):
        """All host threads is not always the fastest for the oracle's many small torch ops (a
        128-core host ran it ~30x slower than 8 threads): time one layer per candidate, keep the best."""
        n = os.cpu_count() or 1
        self.step(1)   # warm-up: first-use conversions are not part of a step
        best, best_t = None, n
        for t in sorted({n, min(n, 32), min(n, 16), min(n, 8)}, reverse=True):
            self.torch.set_num_threads(t)
            v, secs = self.step(1)
            if best is None or v > best:
                best, best_t, self.layer_secs = v, t, self.last_layer_secs
        self.torch.set_num_threads(best_t)

    def layers_for(self, budget_s: float) -> int:
        """How many passes through the (single, repeated) decoder layer fit a CPU-time budget."""
        return int(max(2, min(512, budget_s / max(self.layer_secs, 1e-3))))

    def step(self, n_layers_sample: int):
        """Returns (tokens_per_s extrapolated to 32 layers, seconds spent)."""
        t0 = time.perf_counter()
        y = self.x
        for _ in range(n_layers_sample):
            y = self.ollama.decoder_layer(y, self.pos, self.layer, self.cfg, self.cos_sin, self.kc,
                                          self.vc, self.slots, self.meta)
        t_layers = time.perf_counter() - t0
        t1 = time.perf_counter()
        logits = self.lm_head(self.ops.rms_norm(y, self.fn, self.cfg.rms_eps))
        _ = logits.argmax(-1)
        t_head = time.perf_counter() - t1
        step_s = t_layers / n_layers_sample * 32 + t_head
        self.last_layer_secs = t_layers / n_layers_sample
        return self.B / step_s, t_layers + t_head


def cpu_decode_sample(a, budget_s: float = 30.0, seed: int = 0):
    c = CpuDecodeSample(a, seed)
    n_layers = c.layers_for(budget_s)
    v, secs = c.step(n_layers)
    return v, secs, c.torch.get_num_threads(), n_layers, c.B


def cpu_config0(runs: int = 3, seed: int = 0):
    """BASELINE.json configs[0] — the reference's only CPU-runnable case (gpt2-124M fp32, batch 1,
    8-token prompt, 32 new tokens, greedy; examples/cpu_offline_inference.py) restated in
    oracle/gpt2.py with random-init weights, timed on this box's host cores: median of `runs`.
    A reported baseline beside the GPU numbers, not a target."""
    try:
        import torch
        from oracle import gpt2
        threads = torch.get_num_threads()
        torch.set_num_threads(min(os.cpu_count() or 1, 16))    # small matrices: more threads only add sync
        m = gpt2.init_gpt2(seed)
        prompt = torch.randint(0, 50257, (8,), generator=torch.Generator().manual_seed(seed))
        res = sorted((gpt2.generate(m, prompt, 32) for _ in range(runs)), key=lambda r: r["decode_tok_s"])
        r = res[len(res) // 2]
        out = {"workload": "gpt2-124M fp32 offline generate on CPU, batch 1, 8-token prompt, 32 new tokens",
               "decode_tokens_per_s": r["decode_tok_s"], "ttft_ms": 1e3 * r["ttft_s"],
               "cores": torch.get_num_threads(), "runs": runs, "kind": "port"}
        torch.set_num_threads(threads)
        return out
    except Exception as e:  # noqa: BLE001  (a side figure: never cost the bench line)
        return {"unavailable": f"{type(e).__name__}: {e}"}


def run_reference(a, rank):
    if rank != 0:
        return
    if a.model != "llama3-8b":
        print(json.dumps({"impl": "reference", "unavailable": "the CPU arm is sized for the llama3-8b "
                          "configuration the metric is quoted on"}), flush=True)
        return
    c = CpuDecodeSample(a, 0)
    cores = c.torch.get_num_threads()
    vals, secs = [], []
    for i in range(a.warmup + a.steps):
        v, s = c.step(1)
        if i >= a.warmup:
            vals.append(v)
            secs.append(s)
    vals.sort()
    secs.sort()
    v = vals[len(vals) // 2]
    world = int(os.environ.get("WORLD_SIZE", "1"))
    sample = (f"EXTRAPOLATED: each timed step runs {c.B} of the {a.batch} sequences (kv_len {a.seqlen}) "
              "through 1 of the 32 oracle decoder layers + final norm + bf16 lm_head "
              f"({secs[len(secs) // 2]:.2f} s of CPU work per step on {cores} threads, the fastest of the "
              "thread counts {all, 32, 16, 8} timed at start-up — the same rule as the main arm's "
              "cpu_baseline); value = sampled sequences / (layer time x 32 + head time), i.e. the "
              "tokens/s the CPU path would sustain on the sampled sequences; median over steps")
    out = {"impl": "reference", "metric": METRIC, "value": v, "unit": UNIT, "n_gpus": a.gpus,
           "steps": a.steps, "warmup": a.warmup,
           # the time a timed step of THIS arm really took (the bounded sample), not the extrapolation
           "ms_per_step": 1000.0 * secs[len(secs) // 2],
           "higher_is_better": True, "scaling": "strong", "vs_baseline": None, "dtype": "bf16",
           "data": "synthetic",
           "config": {"workload": workload_name(a, world), "global_batch": a.batch, "seq_len": a.seqlen,
                      "parallelism": f"tp{world}", "layers": 32},
           "extrapolation": {"layers_run": 1, "layers_total": 32, "sequences_run": c.B,
                             "sequences_total": a.batch,
                             "full_step_ms_extrapolated": 1000.0 * c.B / v},
           "cpu_baseline": {"value": v, "unit": UNIT, "cores": cores, "kind": "port",
                            "sample": sample, "config0": cpu_config0()},
           "e2e": {"value": v, "unit": UNIT, "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
           "gpu_launches": 0}
    print(json.dumps(out), flush=True)


# --------------------------------------------------------------------------------------
# B200 arm
# --------------------------------------------------------------------------------------
def run_b200(a, rank, world, local_rank):
    import numpy as np
    import torch
    import torch.distributed as dist

    from scalellm_b200 import kernels
    from scalellm_b200.decode_step import (BlockPool, GraphedStep, LlamaArgs, LlamaDecoder,
                                           StepBuffers, build_decode_batch)
    from scalellm_b200.layers import QuantArgs
    from scalellm_b200.model_parallel import ParallelArgs, ProcessGroup

    torch.cuda.set_device(local_rank)
    dev = torch.device("cuda", local_rank)
    pg = None
    if world > 1:
        dist.init_process_group("nccl", device_id=dev)
        pg = ProcessGroup(rank, world, dev)
    pa = ParallelArgs(rank, world, pg)

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    def max_over_ranks(x: float) -> float:
        if world == 1:
            return x
        t = torch.tensor([x], dtype=torch.float64, device=dev)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        return float(t.item())

    args = LlamaArgs.llama3_70b() if a.model == "llama3-70b" else LlamaArgs.llama3_8b()
    if a.layers is not None:
        args.n_layers = a.layers
    a.layers = args.n_layers
    qa = QuantArgs(quant_method="" if a.quant == "none" else a.quant, bits=4, group_size=128,
                   is_sym=(a.quant == "gptq"))
    model = LlamaDecoder(args, qa, pa, dev)
    model.init_random(seed=0)

    B, S, bs = a.batch, a.seqlen, a.block_size
    total_steps = a.warmup + a.steps
    cap = S + 2 * total_steps + 8              # room for the e2e loop to grow every sequence
    blocks_per_seq = (cap + bs - 1) // bs
    n_blocks = B * blocks_per_seq + 16
    pool = BlockPool(n_blocks, bs, seed=2)
    for _ in range(B):
        pool.add_sequence(cap)
    model.alloc_kv(n_blocks, bs, randomize=True, seed=1)
    bufs = StepBuffers(dev, B, B, B * blocks_per_seq)
    hb = build_decode_batch(pool, [S] * B, [1] * B, args.vocab_size)
    hb.kv_max = cap                            # graph is captured for the longest kv it will see

    # ---- launches per step (claimed gpu_launches) --------------------------------
    tokens, positions, params = bufs.upload(hb)
    kernels.launch_count_reset()
    _ = model(tokens, positions, params, greedy=True)
    torch.cuda.synchronize()
    launches_per_step = kernels.launch_count()

    use_graph = not a.no_graph
    step = None
    if use_graph:
        try:
            step = GraphedStep(model, bufs, hb, greedy=True)
        except Exception as e:  # e.g. a collective that cannot be captured
            if rank == 0:
                print(f"[bench] CUDA graph capture failed ({type(e).__name__}: {e}); eager", file=sys.stderr)
            use_graph = False

    def one_step():
        if use_graph:
            return step.replay()
        return model(tokens, positions, params, greedy=True)

    sampler = ClockSampler(local_rank) if rank == 0 else None

    # ---- device-timed value: inputs resident, K replays --------------------------
    for _ in range(max(a.warmup, 3)):
        one_step()
    barrier()
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    t_w0 = time.perf_counter()
    ev0.record()
    for _ in range(a.steps):
        one_step()
    ev1.record()
    barrier()
    t_w1 = time.perf_counter()
    ms_step = max_over_ranks(ev0.elapsed_time(ev1) / a.steps)
    value = B / (ms_step / 1000.0)

    # ---- end-to-end: host metadata + pinned H2D + step + D2H of the sampled tokens ----
    out_host = torch.empty(B, dtype=torch.int64, pin_memory=True)
    kv = S

    def e2e_step(kv_now):
        hbn = build_decode_batch(pool, [kv_now] * B, [1] * B, args.vocab_size, seed=kv_now)
        hbn.kv_max = cap
        nonlocal tokens, positions, params
        tokens, positions, params = bufs.upload(hbn)
        nxt = one_step()
        out_host.copy_(nxt, non_blocking=True)
        torch.cuda.current_stream().synchronize()
        return hbn

    for _ in range(max(a.warmup, 3)):
        kv += 1
        last = e2e_step(kv)
    barrier()
    t0 = time.perf_counter()
    for _ in range(a.steps):
        kv += 1
        last = e2e_step(kv)
    barrier()
    t_e2e_end = time.perf_counter()
    e2e_s = max_over_ranks((t_e2e_end - t0) / a.steps)
    e2e_val = B / e2e_s
    h2d = bufs.h2d_bytes(last)
    d2h = B * 8

    # ---- roofline of the dominant kernel (paged attention), timed alone -------------
    roof = attention_roofline(model, params, hb, a, dev, world)
    gemm = gemm_roofline(model, a, dev) if a.quant != "none" else None

    clocks = None
    if sampler:
        time.sleep(0.15)
        # under load from the first device-timed step to the last end-to-end step (same graph
        # replayed back to back): a 100 ms nvidia-smi period needs that long for a real median
        clocks = ClockSampler.summarise(sampler.window(t_w0, t_e2e_end))
        sampler.stop()

    # p50 time to first token (the metric's second half): every rank runs the same deterministic
    # request list (the collectives inside need all of them), rank 0 reports
    ttft = "skipped (--no-ttft)"
    if not a.no_ttft:
        try:
            ttft = measure_ttft(model, pool, args, dev, chunk=a.ttft_chunk, n_req=8, use_graph=use_graph)
        except Exception as e:  # noqa: BLE001  (never cost the bench line)
            ttft = f"failed: {type(e).__name__}: {e}"
        barrier()

    cpu = None
    if rank == 0 and world == 1 and not a.skip_cpu_baseline and a.model == "llama3-8b":
        v, secs, cores, n_layers, n_seq = cpu_decode_sample(a)
        cpu = {"value": v, "unit": UNIT, "cores": cores, "kind": "port",
               "sample": f"{n_seq} of the {a.batch} sequences through {n_layers} passes of an oracle decoder layer + "
                         f"lm_head at the full kv_len ({secs:.1f} s of CPU work on {cores} threads, the "
                         "fastest of the thread counts tried), time extrapolated to 32 layers",
               "config0": cpu_config0()}

    kv_gb = 2 * B * S * max(1, args.n_kv_heads // world) * args.head_dim * 2 * args.n_layers / 1e9
    wbytes = 0.5 + 2.5 / 128 if a.quant != "none" else 2.0      # int4 + scales + zeros @ g128
    lin_params = args.hidden_size * ((args.n_heads + 2 * args.n_kv_heads) * args.head_dim +
                                     args.n_heads * args.head_dim + 3 * args.intermediate_size)
    w_gb = (args.n_layers * lin_params * wbytes + args.vocab_size * args.hidden_size * 2) / world / 1e9
    l2_policy = f"inputs larger than L2 ({kv_gb:.1f} GB KV + {w_gb:.1f} GB weights per step" + \
                (" and GPU)" if world > 1 else ")")
    # the whole step against the HBM roofline: every byte the step has to read once (KV of all layers +
    # linear weights + lm_head), per rank, over the device-timed step
    peak_gbs, peak_src = _peaks()
    step_bytes = (kv_gb + w_gb) * 1e9
    step_roof = {"bound": "hbm", "algorithmic_bytes_per_rank": step_bytes,
                 "achieved": step_bytes / (ms_step * 1e-3) / 1e9, "peak": peak_gbs, "unit": "GB/s",
                 "frac": step_bytes / (ms_step * 1e-3) / 1e9 / peak_gbs, "peak_source": peak_src,
                 "what": "whole decode step: KV read + linear weights + lm_head, per rank"}
    if rank == 0:
        out = {"metric": METRIC, "value": value, "unit": UNIT, "n_gpus": world, "steps": a.steps,
               "warmup": a.warmup, "ms_per_step": ms_step, "higher_is_better": True,
               "scaling": "strong", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
               "config": {"workload": workload_name(a, world), "global_batch": B, "seq_len": S,
                          "parallelism": f"tp{world}", "layers": a.layers,
                          "cuda_graph": use_graph,
                          "l2_policy": l2_policy,
                          "ttft": ttft},
               "e2e": {"value": e2e_val, "unit": UNIT, "h2d_bytes_per_step": h2d,
                       "d2h_bytes_per_step": d2h},
               "gpu_launches": launches_per_step * a.steps, "clocks": clocks, "roofline": roof,
               "roofline_step": step_roof, "roofline_w4a16_gemm": gemm, "vs_ref_kernel": _vs_ref_kernel(roof, gemm, a, world),
               "cpu_baseline": cpu}
        print(json.dumps(out), flush=True)
    if world > 1:
        # Tear-down of NCCL communicators that were captured into CUDA graphs can block for
        # minutes; every rank has reported (rank 0 printed), so synchronise and leave hard.
        try:
            dist.barrier()
            torch.cuda.synchronize()
        finally:
            sys.stdout.flush()
            sys.stderr.flush()
            os._exit(0)


def _peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        try:
            return float(json.load(open(p))["hbm_gbs"]), "measured (MEASURED_PEAKS.json, burst copy)"
        except Exception:
            pass
    return 6650.0, "fallback (B200_PROFILING.md)"


def measure_ttft(model, pool, args, dev, n_req: int = 16, chunk: int = 128, seed: int = 4,
                 use_graph: bool = True):
    """Unloaded time-to-first-token: one request at a time, prompt length ~ U[128, 2048] (SURVEY
    §8d traffic shape), chunked prefill with a `chunk`-token budget through the same operator entry
    points as the decode step (attention: the tcgen05 prefill kernel for q_len * group >= 64 rows).
    TTFT = host time from the request's arrival (before its first metadata build) to its first
    generated token being on the host.  Reuses sequence 0's KV blocks of the pool."""
    import numpy as np
    import torch
    from scalellm_b200 import kernels
    from scalellm_b200.decode_step import StepBuffers, build_decode_batch, prefill_chunks
    from scalellm_b200.decode_step import GraphedStep
    rng = np.random.default_rng(seed)
    cap_tokens = pool.n_blocks_of(0) * pool.block_size
    lens = [int(min(x, cap_tokens)) for x in rng.integers(128, 2049, size=n_req)]
    bufs = StepBuffers(dev, chunk, 1, pool.n_blocks_of(0))
    out_host = torch.empty(1, dtype=torch.int64, pin_memory=True)
    # full chunks replay ONE captured graph (the reference captures its decode batch sizes the same
    # way, model_runner.cpp:141-210; the metadata lives in the static buffers, the scalars baked in
    # are the chunk length and the largest kv_len); the ragged last chunk runs eagerly
    graph = None
    if use_graph:
        hb0 = build_decode_batch(pool, [chunk], [chunk], args.vocab_size, seed=seed)
        hb0.kv_max = cap_tokens
        sel_last = torch.tensor([chunk - 1], device=dev)
        graph = GraphedStep(model, bufs, hb0, greedy=True, last_token_idxes=sel_last)
    times = []
    for i, P in enumerate([lens[0]] + lens):            # first request = warm-up, not recorded
        t0 = time.perf_counter()
        sched = prefill_chunks(P, chunk)
        for ci, (q_len, kv_len) in enumerate(sched):
            hb = build_decode_batch(pool, [kv_len], [q_len], args.vocab_size, seed=seed + ci)
            tokens, positions, params = bufs.upload(hb)
            last = ci == len(sched) - 1
            if graph is not None and q_len == chunk:
                ids = graph.replay()
            else:
                sel = torch.tensor([q_len - 1], device=dev) if last else torch.zeros(0, dtype=torch.int64, device=dev)
                ids = model(tokens, positions, params, last_token_idxes=sel, greedy=True)
            if last:
                out_host.copy_(ids, non_blocking=True)
        torch.cuda.current_stream().synchronize()
        if i > 0:
            times.append((time.perf_counter() - t0) * 1e3)
    times.sort()
    return {"p50_ms": times[len(times) // 2], "min_ms": times[0], "max_ms": times[-1],
            "requests": n_req, "prompt_len": "U[128,2048]", "chunk_tokens": chunk,
            "kernels": ("decode path (the stream attention kernel with q_len = chunk rows; B200_ATTN_PREFILL=0)"
                        if os.environ.get("B200_ATTN_PREFILL") == "0" else
                        "tcgen05 prefill attention (csrc/prefill_attn.cu); linears: " +
                        ("the streaming int4 kernel in 128-row passes"
                         if chunk <= 256 or os.environ.get("B200_W4_PREFILL_DENSE", "1") == "0" else
                         "int4 -> bf16 dequant (ours, bit-exact) + library bf16 GEMM above 256 rows, the streaming "
                         "int4 kernel below")),
            "load": "unloaded (one request at a time); full chunks replay a CUDA graph, the ragged last chunk is eager"}


def _traffic(name):
    """DRAM read+write bytes per launch of the kernel, from the committed `ncu --set full` capture
    (profiles/traffic.json, written by tools/ncu_summary.py); None if no capture is committed."""
    p = os.path.join(ROOT, "profiles", "traffic.json")
    try:
        return float(json.load(open(p))[name]["dram_bytes_per_launch"])
    except Exception:
        return None


def _vs_ref_kernel(roof, gemm, a, world):
    """Our live kernel timings beside the reference's own kernels (sm80-era, recompiled for
    sm_100a) as measured on a B200 by tools/attn_bench.py / tools/w4_ref_bench.py on the same
    shapes (profiles/ref_ab.json, profiles/r02_ref_ab.md).  Only for the configuration those
    were taken on: Llama-3-8B, batch 64, kv 2048, block_size 8, one GPU."""
    if world != 1 or a.model != "llama3-8b" or a.batch != 64 or a.seqlen != 2048 or a.block_size != 8:
        return None
    try:
        ref = json.load(open(os.path.join(ROOT, "profiles", "ref_ab.json")))
    except Exception:
        return None
    out = {"source": ref.get("source")}
    if roof:
        out["attention"] = {"reference_us": ref["attention_us"], "ours_us": roof["us_per_launch"],
                            "speedup": ref["attention_us"] / roof["us_per_launch"]}
    if gemm:
        ours = sum(v["us"] for v in gemm["per_proj"].values())
        theirs = sum(ref["marlin_us"][k] for k in gemm["per_proj"])
        out["w4a16_gemms_per_layer"] = {"reference_us": theirs, "ours_us": ours, "speedup": theirs / ours}
    return out


def attention_roofline(model, params, hb, a, dev, world):
    import torch
    from scalellm_b200 import kernels
    H, Hkv, D = model.H, model.Hkv, model.args.head_dim
    B, S = a.batch, a.seqlen
    q = torch.randn(B, H, D, device=dev).to(torch.bfloat16)
    out = torch.empty_like(q)
    caches = model.kv_caches
    sm_scale = D ** -0.5

    def launch(c):
        kernels.paged_kv_varlen_mha(out, q, c.key_cache, c.value_cache, params.q_cu_seq_lens,
                                    params.kv_cu_seq_lens, params.block_tables,
                                    params.cu_block_lens, None, c.block_size(), 1, hb.kv_max,
                                    sm_scale, 0.0, -1)

    for c in caches[:4]:
        launch(c)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    reps = 3
    e0.record()
    for _ in range(reps):
        for c in caches:           # rotating over all layers: every launch reads cold HBM
            launch(c)
    e1.record()
    torch.cuda.synchronize()
    n = reps * len(caches)
    ms = e0.elapsed_time(e1) / n                     # includes the split-KV combine launch
    kv_now = int(params.kv_cu_seq_lens[1].item())
    alg_bytes = 2 * B * kv_now * Hkv * D * 2 + 2 * B * H * D * 2   # K+V read, q read + o write
    peak, src = _peaks()
    ach = alg_bytes / (ms * 1e-3) / 1e9
    return {"kernel": "paged_attn_persist_kernel(+combine)", "bound": "hbm", "achieved": ach,
            "peak": peak, "unit": "GB/s", "frac": ach / peak,
            # the committed ncu capture is of the 1-GPU launch (8 kv heads): no figure for TP shards
            "traffic": _traffic("paged_attn") if world == 1 else None,
            "peak_source": src, "us_per_launch": ms * 1e3, "algorithmic_bytes": alg_bytes,
            "launches_timed": n}


def _time_graphed(fn, reps: int = 3) -> float:
    """ms per replay of `fn` captured into a CUDA graph (no host launch cost in the number)."""
    import torch
    torch.cuda.synchronize()
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        fn()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        fn()
    g.replay()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(reps):
        g.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / reps


def gemm_roofline(model, a, dev):
    """Per-projection W4A16 GEMM launch time, rotating over the layers' weights so they stream
    from HBM.  The launches are replayed from a CUDA graph, as in the decode step: issued from
    Python one by one the three small projections are bound by the host's launch rate, not by the
    kernel (that eager figure is kept as `us_eager`)."""
    import torch
    from scalellm_b200 import kernels
    peak, src = _peaks()
    res = {}
    x_by_k = {}
    layers = model.layers
    for name in ("qkv", "o", "gate_up", "down"):
        mods = [L[name] for L in layers]
        K, N = mods[0].K, mods[0].N
        x = x_by_k.setdefault(K, torch.randn(a.batch, K, device=dev).to(torch.bfloat16))

        def sweep():   # the GEMM launch alone: fp32 stream-K partials out, consumer reduces
            for m in mods:
                kernels.w4a16_gemm_splitk(x, m.packed, N, 128)

        for m in mods[:2]:
            kernels.w4a16_gemm_splitk(x, m.packed, N, 128)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(3):
            sweep()
        e1.record()
        torch.cuda.synchronize()
        ms_eager = e0.elapsed_time(e1) / (3 * len(mods))
        ms, timing = ms_eager, "eager launches"
        try:
            ms_graph = _time_graphed(sweep) / len(mods)
            if 0.0 < ms_graph <= ms_eager * 1.05:
                ms, timing = ms_graph, "CUDA graph replay"
        except Exception as e:  # noqa: BLE001  (keep the eager figure; never cost the bench line)
            timing = f"eager launches (graph capture failed: {type(e).__name__})"
        alg = mods[0].packed.numel() + 2 * a.batch * (K + N)
        ach = alg / (ms * 1e-3) / 1e9
        res[name] = {"K": K, "N": N, "us": ms * 1e3, "us_eager": ms_eager * 1e3, "timing": timing,
                     "achieved": ach, "frac": ach / peak,
                     "tflops": 2.0 * a.batch * K * N / (ms * 1e-3) / 1e12}
    tot_b = sum((model.layers[0][n].packed.numel()) for n in res)
    tot_t = sum(v["us"] for v in res.values())
    return {"bound": "hbm", "unit": "GB/s", "peak": peak, "peak_source": src, "per_proj": res,
            "achieved": tot_b / (tot_t * 1e-6) / 1e9, "frac": tot_b / (tot_t * 1e-6) / 1e9 / peak}


def main():
    a = parse()
    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if a.impl == "reference":
        run_reference(a, rank)
        return
    if a.arch == "kigalix":
        from scalellm_b200 import arch_bench
        arch_bench.run(a)
        return
    if a.arch == "zomurax":
        from scalellm_b200 import arch_bench
        arch_bench.run_zomurax(a)
        return
    if a.arch == "fesupel":
        from scalellm_b200 import arch_bench
        arch_bench.run_fesupel(a)
        return
    if a.arch == "gugalorn":
        from scalellm_b200 import arch_bench
        arch_bench.run_gugalorn(a)
        return
    if a.arch == "palulorn":
        from scalellm_b200 import arch_bench
        arch_bench.run_palulorn(a)
        return
    if a.arch == "pokadra":
        from scalellm_b200 import arch_bench
        arch_bench.run_pokadra(a)
        return
    if world != a.gpus and world == 1 and a.gpus > 1:
        print(f"[bench] --gpus {a.gpus} needs torchrun with {a.gpus} ranks; running 1", file=sys.stderr)
    run_b200(a, rank, world, local_rank)


if __name__ == "__main__":
    main()
