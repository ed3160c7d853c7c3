#!/usr/bin/env python
"""Benchmarks of the GEMM / flash-attention / Qwen3-forward path, one JSON line per run.

    python bench.py --gpus 1 --steps 3 --warmup 3                # headline
    python -m torch.distributed.run --nnodes=1 --nproc-per-node N --master-addr 127.0.0.1 --master-port P \
        bench.py --gpus N --steps K --warmup W
    python bench.py --config 1|2|3|4                             # the other BASELINE configs (one GPU)
    python bench.py --impl reference ...                         # CPU arm: what the reference runs for the path
    python bench.py --model fiferax|molitar [--size 1k|4k]       # a hybrid decoder beside a Qwen3 of equal size (one GPU)

Config 5 (default) and 4: Qwen3-8B / Qwen3-0.6B shaped greedy generation; a "step" is one full generation (prefill,
then CUDA-graph decode steps; the first new token comes out of the prefill); value = tokens (prompt + generated) per
second over the whole job, tensor-parallel over N GPUs for config 5.  Configs 1-3: one kernel (fp32 GEMM 512^3, the
bf16 GEMM sweep, causal GQA flash attention with its decode variant); a step is one launch with an L2 flush before it.
Weights and inputs are seeded random tensors of the configs' shapes (no checkpoints or datasets on this machine).

`value` is timed with CUDA events with everything already on the device; `e2e` is the same work through the public
API with inputs in pinned host memory and results copied back, copies inside the timed region.  `roofline` is the
dominant kernel timed live; for the generation configs `roofline_prefill` and `roofline_decode` add the whole-phase
figures.  `cpu_baseline` is the CPU port of the path timed on a bounded sample on the host cores.  `parity_check`
(generation configs) compares sequence 0's first-token logits with the CPU oracle run at full depth on the same
weights, after the timed region, so a wrong answer at the benchmark's size cannot print a throughput unnoticed.
"""
import argparse
import json
import os
import subprocess
import sys
import threading
import time
import zlib

_JSON_OUT = None  # duplicate of the original stdout, opened in main()

ROOT = os.path.dirname(os.path.abspath(__file__))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

# bounded CPU samples of the generation workloads (roughly 10-30 s of host work on a 16-thread box for cpu_baseline;
# a quarter of that per step for the --impl reference arm, so warm-up + steps stay within a few minutes)
CPU_SAMPLE = {5: dict(sample_layers=4, batch=16, prefill=2048, new_tokens=16),
              4: dict(sample_layers=28, batch=1, prefill=512, new_tokens=32)}
REF_SAMPLE = {5: dict(sample_layers=2, batch=8, prefill=2048, new_tokens=8),
              4: dict(sample_layers=28, batch=1, prefill=512, new_tokens=16)}
MODEL = {5: dict(num_layers=36, hidden=4096, num_q_heads=32, num_kv_heads=8, head_dim=128, intermediate=12288,
                 vocab=151936, eps=1e-6, rope_theta=1e6, tied=False),
         4: dict(num_layers=28, hidden=1024, num_q_heads=16, num_kv_heads=8, head_dim=128, intermediate=3072,
                 vocab=151936, eps=1e-6, rope_theta=1e6, tied=True)}
WORKLOAD = {5: dict(batch=32, prefill=2048, new_tokens=256, seed=4, name="Qwen3-8B"),
            4: dict(batch=1, prefill=512, new_tokens=128, seed=3, name="Qwen3-0.6B")}
METRIC = {1: ("gemm_f32_512_tflops", "TFLOP/s"), 2: ("gemm_bf16_4096x12288x4096_tflops", "TFLOP/s"),
          3: ("flash_attn_causal_b4_h32_s4096_tflops", "TFLOP/s"), 4: ("qwen3_0_6b_tokens_per_s", "tok/s"),
          5: ("qwen3_8b_tokens_per_s", "tok/s")}


def parse_args():
    p = argparse.ArgumentParser()
    p.add_argument("--gpus", type=int, default=1)
    p.add_argument("--steps", type=int, default=3)
    p.add_argument("--warmup", type=int, default=3)
    p.add_argument("--impl", default="ours", choices=["ours", "reference"])
    p.add_argument("--config", type=int, default=5, choices=[1, 2, 3, 4, 5], help="BASELINE.json config (default 5)")
    # workload knobs for debugging only (defaults = the BASELINE config); echoed in `config`
    p.add_argument("--layers", type=int, default=None)
    p.add_argument("--batch", type=int, default=None)
    p.add_argument("--prefill", type=int, default=None)
    p.add_argument("--new-tokens", type=int, default=None)
    p.add_argument("--weights", default="bf16", choices=["bf16", "fp8"],
                   help="config 4/5 only: fp8 = projections and LM head as FP8 E4M3 with per-channel scales (weight-only; "
                        "the arithmetic stays bf16 x bf16 -> f32).  A variant beside the headline, not the headline.")
    p.add_argument("--model", default="qwen3", choices=["qwen3", "fiferax", "molitar"],
                   help="fiferax, molitar: prefill and decode of that decoder and its kernels beside a Qwen3 of equal size (one GPU); "
                        "--size picks the layer sizes, --config does not apply")
    p.add_argument("--size", default="4k", choices=["1k", "4k"])
    p.add_argument("--no-cpu-baseline", action="store_true")
    p.add_argument("--no-verify", action="store_true", help="skip the CPU-oracle check of sequence 0 after the timing")
    return p.parse_args()


def host_threads():
    """Host cores this process may use (torch.distributed.run exports OMP_NUM_THREADS=1, which is not a property of the
    machine: the CPU legs set their thread count from this instead)."""
    try:
        return max(1, len(os.sched_getaffinity(0)))
    except AttributeError:
        return max(1, os.cpu_count() or 1)


def emit(line):
    print(json.dumps(line), file=_JSON_OUT or sys.stdout, flush=True)


# ------------------------------------------------------------------------------------------------ peaks / clocks
def measured_peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        d = json.load(open(path))
        return {"bf16_tflops": d["bf16_tflops"], "bf16_tflops_sustained": d.get("bf16_tflops_sustained") or d["bf16_tflops"],
                "hbm_gbs": d["hbm_gbs"], "source": "measured"}
    return {"bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0, "hbm_gbs": 6650.0, "source": "fallback"}


class ClockSampler:
    """Samples SM clock and throttle reasons of one GPU with nvidia-smi while the timed region runs."""
    FIELDS = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index):
        self.index, self.rows, self.proc = index, [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", str(self.index), f"--query-gpu={self.FIELDS}",
                                          "--format=csv,noheader,nounits", "-lms", "200"], stdout=subprocess.PIPE,
                                         stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def stop(self):
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        time.sleep(0.05)
        mhz = sorted(int(r[0]) for r in self.rows if r and r[0].isdigit())
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = sorted({n for r in self.rows if len(r) >= 6 for n, v in zip(names, r[2:6]) if v.lower().startswith("active")})
        smax = next((int(r[1]) for r in self.rows if len(r) > 1 and r[1].isdigit()), None)
        return {"sm_mhz": mhz[len(mhz) // 2] if mhz else None, "sm_max_mhz": smax, "reasons": reasons,
                "samples": len(mhz)}


# ------------------------------------------------------------------------------------------------ CPU legs
def cpu_generation_rate(cfg_kwargs, sample_layers, batch, prefill, new_tokens):
    """Times the CPU port of the path (oracle.qwen3.OracleQwen3 -- the op sequence HF transformers runs for the
    reference's Qwen3 script, on PyTorch CPU) on `sample_layers` layers of the real shapes and scales the layer time
    to the full depth.  Returns (tok/s for the full-depth model on the sample's batch / prompt, description, threads)."""
    import torch
    from oracle import qwen3 as oq
    torch.set_num_threads(host_threads())
    full_layers = cfg_kwargs["num_layers"]
    sample_layers = min(sample_layers, full_layers)
    kw = dict(cfg_kwargs)
    kw["num_layers"] = sample_layers
    cfg = oq.OracleQwen3Config(**kw)
    # timing does not depend on the values: every tensor is a view into one random block (fast to create)
    H, D = cfg.hidden, cfg.head_dim
    biggest = max(cfg.vocab * H, cfg.intermediate * H)
    block = (torch.randn(biggest // 64 + 1, generator=torch.Generator().manual_seed(4)) * 0.02).bfloat16().repeat(64)

    def view(*shape):
        n = 1
        for s in shape:
            n *= s
        return block[:n].view(*shape)

    sd = {"model.embed_tokens.weight": view(cfg.vocab, H), "model.norm.weight": torch.ones(H, dtype=torch.bfloat16)}
    if not cfg.tied:
        sd["lm_head.weight"] = view(cfg.vocab, H)
    for i in range(sample_layers):
        p = f"model.layers.{i}."
        sd[p + "self_attn.q_proj.weight"] = view(cfg.num_q_heads * D, H)
        sd[p + "self_attn.k_proj.weight"] = view(cfg.num_kv_heads * D, H)
        sd[p + "self_attn.v_proj.weight"] = view(cfg.num_kv_heads * D, H)
        sd[p + "self_attn.o_proj.weight"] = view(H, cfg.num_q_heads * D)
        sd[p + "mlp.gate_proj.weight"] = view(cfg.intermediate, H)
        sd[p + "mlp.up_proj.weight"] = view(cfg.intermediate, H)
        sd[p + "mlp.down_proj.weight"] = view(H, cfg.intermediate)
        for n in ("self_attn.q_norm.weight", "self_attn.k_norm.weight"):
            sd[p + n] = torch.ones(D, dtype=torch.bfloat16)
        for n in ("input_layernorm.weight", "post_attention_layernorm.weight"):
            sd[p + n] = torch.ones(H, dtype=torch.bfloat16)
    ids = torch.randint(0, cfg.vocab, (batch, prefill), generator=torch.Generator().manual_seed(5))

    def run(layers_cfg):
        m = oq.OracleQwen3(layers_cfg, sd)
        t0 = time.perf_counter()
        m.generate(ids, new_tokens)
        return time.perf_counter() - t0

    zero = oq.OracleQwen3Config(**{**kw, "num_layers": 0})
    run(zero)                      # warm-up of the head path (thread pools, allocator)
    t_head = run(zero)             # embedding + final norm + LM head + argmax only
    t_some = run(cfg)
    per_layer = max(t_some - t_head, 0.0) / sample_layers
    t_full = t_head + per_layer * full_layers
    tokens = batch * (prefill + new_tokens)
    desc = (f"{sample_layers} of {full_layers} layers + embedding/LM head timed, layer time scaled to {full_layers}; "
            f"batch {batch}, prefill {prefill}, {new_tokens} greedy tokens; PyTorch CPU bf16, "
            f"{torch.get_num_threads()} threads; measured {t_some:.2f}s (+{t_head:.2f}s head-only)")
    return tokens / t_full, desc, torch.get_num_threads()


def cpu_kernel_rate(config):
    """CPU leg of the single-kernel configs: (value in the config's unit, description, threads, seconds per sample)."""
    import numpy as np
    import torch
    import torch.nn.functional as F
    torch.set_num_threads(host_threads())
    if config == 1:
        # the reference's own CPU matmul for this workload is the test-side triple loop
        # (kernels/teeny-kernels/tests/test_gemm.rs:183-196), restated in C in oracle/teeny_oracle.c: one thread
        from oracle import cpu as oc
        g = torch.Generator().manual_seed(0)
        a, b = torch.randn(512, 512, generator=g).numpy(), torch.randn(512, 512, generator=g).numpy()
        oc.matmul_f32(a, b)
        t0 = time.perf_counter()
        reps = 5
        for _ in range(reps):
            oc.matmul_f32(a, b)
        dt = (time.perf_counter() - t0) / reps
        ta, tb = torch.from_numpy(a), torch.from_numpy(b)
        torch.matmul(ta, tb)
        t0 = time.perf_counter()
        for _ in range(50):
            torch.matmul(ta, tb)
        dt2 = (time.perf_counter() - t0) / 50
        fl = 2 * 512 ** 3
        return fl / dt / 1e12, (f"sequential f32 triple loop (the reference's test-side matmul_reference restated in C), "
                                f"512^3, {reps} runs; torch.matmul f32 on {torch.get_num_threads()} threads for comparison: "
                                f"{fl / dt2 / 1e12:.4f} TFLOP/s"), 1, dt
    if config == 2:
        M, N, K = 4096, 12288, 4096
        g = torch.Generator().manual_seed(1)
        x = ((torch.rand(M // 4, K, generator=g) * 2 - 1) * 0.05).bfloat16()
        w = ((torch.rand(N, K, generator=g) * 2 - 1) * 0.05).bfloat16()
        F.linear(x.float(), w.float())
        t0 = time.perf_counter()
        F.linear(x.float(), w.float()).bfloat16()
        dt = time.perf_counter() - t0
        return 2.0 * (M // 4) * N * K / dt / 1e12, (f"F.linear on bf16 inputs up-cast to f32, a quarter of the rows "
                                                     f"({M // 4} x {N} x {K}), {torch.get_num_threads()} threads"), torch.get_num_threads(), dt
    if config == 3:
        B, Hq, Hkv, S, D = 1, 32, 8, 4096, 128
        g = torch.Generator().manual_seed(2)
        q = torch.randn(B, Hq, S, D, generator=g).bfloat16()
        k = torch.randn(B, Hkv, S, D, generator=g).bfloat16()
        v = torch.randn(B, Hkv, S, D, generator=g).bfloat16()
        rep = Hq // Hkv
        t0 = time.perf_counter()
        F.scaled_dot_product_attention(q.float(), k.float().repeat_interleave(rep, 1), v.float().repeat_interleave(rep, 1),
                                       is_causal=True, scale=D ** -0.5).bfloat16()
        dt = time.perf_counter() - t0
        return 0.5 * 4 * B * Hq * S * S * D / dt / 1e12, (f"F.scaled_dot_product_attention (causal, KV heads repeated, f32) on "
                                                          f"batch 1 of 4, {torch.get_num_threads()} threads; causal FLOP count"), torch.get_num_threads(), dt
    raise ValueError(config)


def reference_arm(args):
    """The reference's CPU execution of the path.  Its Qwen3 script runs the traced PyTorch graph on the CPU
    (support/teeny-torch/python/teenygrad/atlas/module.py:42-45) and its only CPU matmul is the test-side triple loop;
    the Rust crates cannot be built here (no cargo, no teenyc), so this times the CPU port of those on a bounded sample
    per step, on every host core.  Under torch.distributed.run only rank 0 works."""
    if int(os.environ.get("RANK", "0")) != 0:
        return
    cfgn = args.config
    vals, desc, threads = [], "", 1
    for i in range(args.warmup + args.steps):
        if cfgn in (4, 5):
            v, desc, threads = cpu_generation_rate(model_kwargs(args), **REF_SAMPLE[cfgn])
        else:
            v, desc, threads, sample_s = cpu_kernel_rate(cfgn)
        if i >= args.warmup:
            vals.append(v)
    value = sum(vals) / len(vals)
    metric, unit = METRIC[cfgn]
    if cfgn in (4, 5):
        s = REF_SAMPLE[cfgn]
        ms = 1000.0 * s["batch"] * (s["prefill"] + s["new_tokens"]) / value
    else:
        ms = 1000.0 * sample_s
    line = {"impl": "reference", "metric": metric, "value": value, "unit": unit, "n_gpus": args.gpus,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": ms,
            "higher_is_better": True, "scaling": "strong", "vs_baseline": None,
            "dtype": "f32" if cfgn == 1 else "bf16", "data": "synthetic",
            "config": workload_config(args, args.gpus),
            "cpu_baseline": {"value": value, "unit": unit, "cores": threads, "kind": "port", "sample": desc},
            "e2e": {"value": value, "unit": unit, "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0}}
    emit(line)


def model_kwargs(args):
    kw = dict(MODEL[args.config])
    if args.layers is not None:
        kw["num_layers"] = args.layers
    return kw


def workload_of(args):
    w = dict(WORKLOAD[args.config])
    for k, a in (("batch", args.batch), ("prefill", args.prefill), ("new_tokens", args.new_tokens)):
        if a is not None:
            w[k] = a
    return w


def workload_config(args, n):
    c = args.config
    if c in (4, 5):
        kw, w = model_kwargs(args), workload_of(args)
        return {"workload": f"{w['name']}-shaped decoder ({kw['num_layers']} layers, hidden {kw['hidden']}, {kw['num_q_heads']} q / "
                            f"{kw['num_kv_heads']} kv heads, head_dim 128, intermediate {kw['intermediate']}, vocab {kw['vocab']}, "
                            f"{'tied' if kw['tied'] else 'untied'} head), random-init bf16 seed {w['seed']}; batch {w['batch']}, "
                            f"prefill {w['prefill']} uniform-random ids, {w['new_tokens']} greedy tokens",
                "baseline_config": c, "global_batch": w["batch"], "seq_len": w["prefill"], "new_tokens": w["new_tokens"],
                "parallelism": f"tp{n}", "l2": "inputs larger than L2 (weights + KV cache stream every step)"
                if c == 5 else "L2 flushed between generations is not needed: 1.2 GB of weights stream every decode step"}
    text = {1: "fp32 GEMM C = A B, A and B 512 x 512 row-major, N(0,1) seed 0",
            2: "bf16 GEMM sweep, fp32 accumulate: N = K = 4096 with M in {1, 16, 128, 4096}, and M = 4096, N = 12288, K = 4096; "
               "U(-1,1) * 0.05 seed 1, row-major A, K-major B; value = the M = 4096, N = 12288 shape",
            3: "causal GQA flash-attention forward, bf16, batch 4, 32 / 8 heads, head_dim 128, sequence 4096, N(0,1) seed 2; "
               "plus the decode variant (1 query token against 4096 cached)"}[c]
    return {"workload": text, "baseline_config": c, "parallelism": "1 GPU",
            "l2": "L2 flushed (256 MB write) before every timed launch; microsecond-scale launches (M <= 128, decode "
                  "attention) replayed from a CUDA graph over rotating input copies larger than L2"}


# ------------------------------------------------------------------------------------------------ single-kernel configs
def kernel_config(args):
    import torch
    from teenygrad_b200 import ops
    from teenygrad_b200._lib import lib
    if args.gpus != 1:
        raise SystemExit("configs 1-3 are single-GPU kernels")
    torch.cuda.set_device(0)
    peaks = measured_peaks()
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    warm = max(args.warmup, 3)

    def timed(fn, steps=args.steps):
        for _ in range(warm):
            fn()
        ts = []
        for _ in range(steps):
            flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        return sum(ts) / len(ts)

    def graph_timed(fns, reps=5):
        """Microsecond-scale kernels: one CUDA graph of launches over rotating copies of their inputs (together larger
        than L2, so every launch streams from HBM and no host launch gap enters); replayed, CUDA events on the replaying
        stream; returns ms per launch."""
        st = torch.cuda.Stream()
        with torch.cuda.stream(st):
            for f in fns:
                f()
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g, stream=st):
                for f in fns:
                    f()
            for _ in range(warm):
                g.replay()
            torch.cuda.synchronize()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            for _ in range(reps):
                g.replay()
            b.record()
            torch.cuda.synchronize()
        return a.elapsed_time(b) / reps / len(fns)

    def e2e_timed(host_inputs, run, out_dev_to_host):
        """inputs from pinned host memory, result read back, all inside the timed region (wall clock around a sync)."""
        def once():
            devs = [h.to("cuda", non_blocking=True) for h in host_inputs]
            out_dev_to_host(run(*devs))
            torch.cuda.current_stream().synchronize()
        for _ in range(2):
            once()
        t0 = time.perf_counter()
        for _ in range(args.steps):
            once()
        return (time.perf_counter() - t0) / args.steps * 1e3

    metric, unit = METRIC[args.config]
    sampler = ClockSampler(0)
    sampler.start()
    lib.teeny_launch_count(1)
    extra = {}
    if args.config == 1:
        g = torch.Generator().manual_seed(0)
        ah, bh = torch.randn(512, 512, generator=g).pin_memory(), torch.randn(512, 512, generator=g).pin_memory()
        a, b = ah.cuda(), bh.cuda()
        c = torch.empty(512, 512, device="cuda")
        sc = ops.matmul_f32_scratch(512, 512, 512)
        ms = timed(lambda: ops.matmul_forward(a, b, out=c, scratch=sc), steps=max(args.steps, 20))   # tensor cores, bf16 x 3
        ms_simt = timed(lambda: ops.matmul_forward(a, b, out=c), steps=max(args.steps, 20))          # CUDA cores
        ms_t = timed(lambda: torch.matmul(a, b, out=c), steps=max(args.steps, 20))
        fl = 2.0 * 512 ** 3
        value = fl / ms / 1e9
        extra["cuda_core_path_tflops"] = fl / ms_simt / 1e9
        ch = torch.empty(512, 512).pin_memory()
        e2e_ms = e2e_timed([ah, bh], lambda x, y: ops.matmul_forward(x, y), lambda o: ch.copy_(o, non_blocking=True))
        h2d, d2h = 2 * 512 * 512 * 4, 512 * 512 * 4
        # three bf16 tensor-core products per f32 product: the bound is a third of the bf16 peak
        peak = peaks["bf16_tflops"] / 3.0
        roof = {"bound": "tensor", "kernel": "f32 GEMM 512^3 on the tensor cores, operands split into bf16 terms (latency-dominated: 2.7e8 FLOP, 3 launches)", "achieved": value, "peak": peak,
                "unit": "TFLOP/s", "frac": value / peak, "peak_source": peaks["source"] + " (burst cuBLAS bf16 / 3: three bf16 products per f32 product)",
                "traffic": None}
        extra["torch_matmul_f32_tflops"] = fl / ms_t / 1e9
        dtype = "f32"
    elif args.config == 2:
        sweep = []
        for (M, N, K) in [(1, 4096, 4096), (16, 4096, 4096), (128, 4096, 4096), (4096, 4096, 4096), (4096, 12288, 4096)]:
            g = torch.Generator(device="cuda").manual_seed(1)
            x = ((torch.rand(M, K, generator=g, device="cuda") * 2 - 1) * 0.05).bfloat16()
            w = ((torch.rand(N, K, generator=g, device="cuda") * 2 - 1) * 0.05).bfloat16()
            y = torch.empty(M, N, dtype=torch.bfloat16, device="cuda")
            if M <= 128:   # tens of microseconds: graph of launches over 24 weight copies (805 MB, L2 is 126 MB)
                ws = [w] + [w.clone() for _ in range(23)]
                ms = graph_timed([(lambda wi=wi: ops.linear_forward(x, wi, out=y)) for wi in ws])
                ms_t = graph_timed([(lambda wi=wi: torch.matmul(x, wi.t(), out=y)) for wi in ws])
                del ws
            else:
                ms = timed(lambda: ops.linear_forward(x, w, out=y), steps=max(args.steps, 10))
                ms_t = timed(lambda: torch.matmul(x, w.t(), out=y), steps=max(args.steps, 10))
            fl, by = 2.0 * M * N * K, 2.0 * (M * K + N * K + M * N)
            hbm_bound = M <= 128  # 2 FLOP per weight byte x M: below ~250 rows the weight read bounds the kernel
            ach = by / ms / 1e6 if hbm_bound else fl / ms / 1e9
            pk = peaks["hbm_gbs"] if hbm_bound else peaks["bf16_tflops"]
            sweep.append({"M": M, "N": N, "K": K, "us": ms * 1e3, "bound": "hbm" if hbm_bound else "tensor",
                          "achieved": ach, "unit": "GB/s" if hbm_bound else "TFLOP/s", "frac": ach / pk,
                          "cublas_us": ms_t * 1e3})
        head = sweep[-1]
        value, ms = head["achieved"], head["us"] / 1e3
        M, N, K = 4096, 12288, 4096
        xh = torch.empty(M, K, dtype=torch.bfloat16).pin_memory()
        yh = torch.empty(M, N, dtype=torch.bfloat16).pin_memory()
        e2e_ms = e2e_timed([xh], lambda xd: ops.linear_forward(xd, w), lambda o: yh.copy_(o, non_blocking=True))
        h2d, d2h = M * K * 2, M * N * 2
        roof = {"bound": "tensor", "kernel": "gemm_bf16_2cta_kernel 4096 x 12288 x 4096", "achieved": value,
                "peak": peaks["bf16_tflops"], "unit": "TFLOP/s", "frac": value / peaks["bf16_tflops"],
                "peak_source": peaks["source"] + " (burst cuBLAS bf16: kernel timed alone)",
                "traffic": 0.99 * 2.0 * (M * K + N * K + M * N),
                "traffic_unit": "bytes per launch (ncu: 231.6 MB on this shape)"}
        extra["sweep"] = sweep
        dtype = "bf16"
    else:
        B, Hq, Hkv, S, D = 4, 32, 8, 4096, 128
        g = torch.Generator(device="cuda").manual_seed(2)
        q = torch.randn(B, Hq, S, D, generator=g, device="cuda").bfloat16()
        k = torch.randn(B, Hkv, S, D, generator=g, device="cuda").bfloat16()
        v = torch.randn(B, Hkv, S, D, generator=g, device="cuda").bfloat16()
        o = torch.empty_like(q)
        ms = timed(lambda: ops.flash_attn_fwd(q, k, v, D ** -0.5, causal=True, out=o), steps=max(args.steps, 10))
        ms_t = timed(lambda: torch.nn.functional.scaled_dot_product_attention(q, k, v, is_causal=True, enable_gqa=True),
                     steps=max(args.steps, 10))
        fl = 0.5 * 4 * B * Hq * S * S * D
        value = fl / ms / 1e9
        q1 = torch.randn(B, Hq, 1, D, generator=g, device="cuda").bfloat16()
        o1 = torch.empty_like(q1)
        sc = torch.empty(lib.teeny_attn_decode_scratch_bytes(B, Hq, D, S), dtype=torch.uint8, device="cuda")
        kvs = [(k, v)] + [(torch.randn_like(k), torch.randn_like(v)) for _ in range(5)]   # 6 x 67 MB of cache
        ms_d = graph_timed([(lambda kk=kk, vv=vv: ops.flash_attn_decode(q1, kk, vv, S, D ** -0.5, out=o1, scratch=sc))
                            for kk, vv in kvs])
        del kvs
        by_d = 2.0 * B * Hkv * S * D * 2
        qh, kh, vh = (t.cpu().pin_memory() for t in (q, k, v))
        oh = torch.empty(B, Hq, S, D, dtype=torch.bfloat16).pin_memory()
        e2e_ms = e2e_timed([qh, kh, vh], lambda a, b, c: ops.flash_attn_fwd(a, b, c, D ** -0.5, causal=True),
                           lambda r: oh.copy_(r, non_blocking=True))
        h2d, d2h = (q.numel() + k.numel() + v.numel()) * 2, q.numel() * 2
        roof = {"bound": "tensor", "kernel": "attention_prefill_kernel B4 H32/8 S4096 causal", "achieved": value,
                "peak": peaks["bf16_tflops"], "unit": "TFLOP/s", "frac": value / peaks["bf16_tflops"],
                "peak_source": peaks["source"] + " (burst cuBLAS bf16: kernel timed alone)",
                "traffic": 453.5e6, "traffic_unit": "bytes per launch (ncu on this shape; 268 MB algorithmic, K/V re-reads that miss L2 on top)"}
        extra["torch_sdpa_tflops"] = fl / ms_t / 1e9
        extra["decode_variant"] = {"us": ms_d * 1e3, "achieved": by_d / ms_d / 1e6, "unit": "GB/s", "bound": "hbm",
                                   "frac": by_d / ms_d / 1e6 / peaks["hbm_gbs"], "bytes": by_d}
        dtype = "bf16"
    launches = int(lib.teeny_launch_count(1))
    clocks = sampler.stop()
    err = lib.teeny_device_error(1)
    if err != 0:
        raise SystemExit(f"device error word {err:#x}")
    line = {"metric": metric, "value": value, "unit": unit, "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
            "warmup_run": warm, "ms_per_step": ms, "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
            "dtype": dtype, "data": "synthetic", "config": workload_config(args, 1),
            "e2e": {"value": value * ms / e2e_ms, "unit": unit, "ms_per_step": e2e_ms, "h2d_bytes_per_step": h2d,
                    "d2h_bytes_per_step": d2h},
            "gpu_launches": launches, "clocks": clocks, "roofline": roof, **extra}
    if not args.no_cpu_baseline:
        v, desc, threads, _ = cpu_kernel_rate(args.config)
        line["cpu_baseline"] = {"value": v, "unit": unit, "cores": threads, "kind": "port", "sample": desc}
    emit(line)


# ------------------------------------------------------------------------------------------------ generation configs
def generation_config(args):
    import torch
    import torch.distributed as dist
    from teenygrad_b200 import ops, qwen3, tp
    from teenygrad_b200._lib import lib

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    if world != args.gpus:
        raise SystemExit(f"--gpus {args.gpus} but WORLD_SIZE={world}: launch with torch.distributed.run")
    torch.cuda.set_device(local)
    dev = torch.device("cuda", local)
    comm = None
    if world > 1:
        dist.init_process_group("nccl", device_id=dev)
        comm = tp.init_comm(rank, world)

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    cfg_kwargs, wl = model_kwargs(args), workload_of(args)
    B, S, NEW, seed = wl["batch"], wl["prefill"], wl["new_tokens"], wl["seed"]
    cfg = qwen3.Qwen3Config(**cfg_kwargs)
    runner = qwen3.Qwen3Runner(cfg, max_batch=B, max_len=S + NEW, max_tokens=B * S, max_new_tokens=NEW,
                               tp_rank=rank, tp_size=world, comm=comm)
    fp8 = args.weights == "fp8"
    qwen3.load_random_weights(runner, seed=seed, fp8=fp8)
    tp_mode = "none" if world == 1 else ("peer-push" if lib.teeny_tp_peer_enabled(comm) else "nccl-allreduce")
    g = torch.Generator().manual_seed(seed)
    prompts_host = torch.randint(0, cfg.vocab, (B, S), generator=g, dtype=torch.int32).pin_memory()
    prompts_dev = prompts_host.to(dev)
    out_host = torch.empty(B, NEW, dtype=torch.int32).pin_memory()
    tokens_per_step = B * (S + NEW)

    def one_generation_device():
        return runner.generate(prompts_dev, NEW, use_graph=True)

    def one_generation_e2e():
        ids = prompts_host.to(dev, non_blocking=True)         # H2D of this step's inputs
        out = runner.generate(ids, NEW, use_graph=True)
        out_host.copy_(out, non_blocking=True)                # D2H of the step's result
        torch.cuda.current_stream().synchronize()

    warm = max(args.warmup, 3)  # timing rule: at least three warm-up generations, whatever was asked
    for _ in range(warm):
        one_generation_device()
    barrier()

    # ---- timed region: device-resident inputs ----
    sampler = ClockSampler(local)
    if rank == 0:
        sampler.start()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    pre = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(args.steps)]
    barrier()
    lib.teeny_launch_count(1)
    e0.record()
    for i in range(args.steps):
        pre[i][0].record()
        runner.prefill(prompts_dev)
        pre[i][1].record()
        for _ in range(NEW - 1):
            runner.decode_step(graph=True)
    e1.record()
    barrier()
    launches = int(lib.teeny_launch_count(1))
    clocks = sampler.stop() if rank == 0 else None
    ms = torch.tensor([e0.elapsed_time(e1), sum(a.elapsed_time(b) for a, b in pre)], device=dev, dtype=torch.float64)
    if world > 1:
        dist.all_reduce(ms, op=dist.ReduceOp.MAX)
    total_ms, prefill_ms = float(ms[0]), float(ms[1])
    err = lib.teeny_device_error(1)
    if err != 0:
        raise SystemExit(f"device error word {err:#x} after the timed region")
    ids_crc = zlib.crc32(runner.history()[:NEW].t().contiguous().cpu().numpy().tobytes())
    first_crc = zlib.crc32(runner.history()[0].contiguous().cpu().numpy().tobytes())

    # ---- end to end through the public API, host buffers ----
    one_generation_e2e()
    barrier()
    t0 = time.perf_counter()
    for _ in range(args.steps):
        one_generation_e2e()
    barrier()
    e2e_s = torch.tensor([time.perf_counter() - t0], device=dev, dtype=torch.float64)
    if world > 1:
        dist.all_reduce(e2e_s, op=dist.ReduceOp.MAX)

    # ---- dominant kernel: the tcgen05 GEMM on this run's prefill shapes (per rank), CUDA events, timed alone ----
    peaks = measured_peaks()
    T, H, I = B * S, cfg.hidden, cfg.intermediate
    qkv_n = (cfg.num_q_heads + 2 * cfg.num_kv_heads) * 128
    shapes = [(T, qkv_n // world, H), (T, H, cfg.num_q_heads * 128 // world), (T, 2 * I // world, H), (T, H, I // world)]
    flops = gemm_ms = gemm_bytes = 0.0
    x = torch.empty(T, max(I // world, H), dtype=torch.bfloat16, device=dev).normal_(0, 0.05)
    wbuf = torch.empty(max(2 * I * H // world, H * qkv_n), dtype=torch.bfloat16, device=dev).normal_(0, 0.02)
    ybuf = torch.empty(T * max(2 * I // world, qkv_n), dtype=torch.bfloat16, device=dev)
    for (m, n, k) in shapes:
        xv, wv, yv = x[:, :k], wbuf[:n * k].view(n, k), ybuf[:m * n].view(m, n)
        # "alone" as the burst peak it is divided by was measured: from an idle GPU, not on the heels of seconds of
        # power-capped generation (the in-step figure against the sustained peak is roofline_prefill)
        torch.cuda.synchronize()
        time.sleep(1.0)
        for _ in range(2):
            ops.linear_forward(xv, wv, out=yv)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(3):
            ops.linear_forward(xv, wv, out=yv)
        b.record()
        torch.cuda.synchronize()
        gemm_ms += a.elapsed_time(b) / 3
        flops += 2.0 * m * n * k
        gemm_bytes += 2.0 * (m * k + n * k + m * n)
    achieved = flops / (gemm_ms * 1e-3) / 1e12
    del x, wbuf, ybuf

    # ---- parity: sequence 0's first-token logits against the CPU oracle at full depth, same weights ----
    parity = None
    if not args.no_verify:
        runner.prefill(prompts_dev)
        row = runner.logits()[0].clone()
        if world > 1:
            parts = [torch.empty_like(row) for _ in range(world)]
            dist.all_gather(parts, row)
            row = torch.cat(parts)
        torch.cuda.synchronize()
        if rank == 0:
            from oracle import qwen3 as oq
            torch.set_num_threads(host_threads())
            t0 = time.perf_counter()
            sd = {name: t.cpu() for name, t in qwen3.random_weights_device(cfg, seed, dev)}
            if fp8:  # the oracle sees the dequantised weights (f32) and multiplies bf16 activations with them in f32
                from teenygrad_b200 import quant
                for name in list(sd):
                    if sd[name].dim() >= 2 and name != "model.embed_tokens.weight":
                        sd[name] = quant.quantize_fp8(sd[name]).dequantize()
            oracle = oq.OracleQwen3(oq.OracleQwen3Config(**cfg_kwargs), sd, f32_twin=fp8)
            want = oracle.forward(prompts_host[:1].long())[0].float()
            # The 2e-2 bar is a per-kernel bar (the GPU tests hold every kernel and one whole layer to it).  Through a
            # deep stack two correct bf16 evaluations drift apart: the oracle's own f32-accumulating twin (same graph,
            # same rounding points, another summation order) measures by how much at this depth, and the GPU must be
            # as close to the oracle as that twin is (x 1.5), or within 2e-2.
            if fp8:
                # here the oracle itself is the f32-accumulating evaluation (bf16 activations x f32 weights); its twin is
                # the plain bf16 evaluation on the same weights rounded to bf16, which is what a large prefill computes
                sd = {k: v.to(torch.bfloat16) for k, v in sd.items()}
            twin = oq.OracleQwen3(oq.OracleQwen3Config(**cfg_kwargs), sd, f32_twin=not fp8).forward(prompts_host[:1].long())[0].float()
            got = row.float().cpu()
            scale = float(want.abs().max())
            rel = float((got - want).abs().max()) / scale
            floor = float((twin - want).abs().max()) / scale
            bar = max(2e-2, 1.5 * floor)
            gi, wi = int(torch.argmax(got)), int(torch.argmax(want))
            gap = float(want.max() - want[gi]) / scale
            parity = {"what": "sequence 0 of the batch, first generated token, all layers, against oracle/qwen3.py on the host",
                      "logits_rel_err": rel, "oracle_vs_its_f32_twin": floor, "bar": bar, "token": gi, "oracle_token": wi,
                      "token_ok": gi == wi or gap < bar, "ok": rel < bar and (gi == wi or gap < bar),
                      "seconds": time.perf_counter() - t0}
            del sd, oracle

    if rank != 0:
        if world > 1:
            dist.barrier()
            dist.destroy_process_group()
        return

    steps = args.steps
    ov = os.environ.get("TEENY_TP_OVERLAP")  # the library's default: overlapped from 8 ranks on
    prefill_overlap = world > 1 and ((ov == "1") if ov else world >= 8)
    value = tokens_per_step * steps / (total_ms * 1e-3)
    decode_ms = total_ms - prefill_ms
    step_ms = decode_ms / steps / max(NEW - 1, 1)
    L, D = cfg.num_layers, 128
    # algorithmic work per GPU: matmul parameters (2 FLOP / 2 bytes each), causal attention, KV-cache read at the mean length
    layer_params = H * qkv_n + cfg.num_q_heads * D * H + 3 * I * H
    head_params = cfg.vocab * H
    prefill_flop = (2.0 * L * layer_params * T + 2.0 * head_params * B + L * 2.0 * B * cfg.num_q_heads * S * S * D) / world
    mean_len = S + (NEW - 1) / 2.0 + 0.5
    wbytes = 1.0 if fp8 else 2.0  # bytes per matmul parameter as it is streamed in decode
    decode_bytes = (wbytes * (L * layer_params + head_params) + L * 2.0 * B * cfg.num_kv_heads * D * 2.0 * mean_len) / world
    metric, unit = METRIC[args.config]
    line = {
        "metric": metric, "value": value, "unit": unit, "n_gpus": world, "steps": steps, "warmup": args.warmup,
        "warmup_run": warm, "ms_per_step": total_ms / steps, "higher_is_better": True, "scaling": "strong",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {**workload_config(args, world), "weights": "fp8-e4m3, per-channel scales, weight-only" if fp8 else "bf16",
                   "tp_decode_reduction": tp_mode, "tp_prefill_reduction":
                   "none" if world == 1 else ("nccl-allreduce, overlapped with the other half-batch's compute"
                                              if prefill_overlap else "nccl-allreduce")},
        "phases": {"prefill_ms": prefill_ms / steps, "decode_ms": decode_ms / steps,
                   "prefill_tok_s": B * S * steps / (prefill_ms * 1e-3),
                   "decode_tok_s": B * (NEW - 1) * steps / max(decode_ms * 1e-3, 1e-9),
                   "decode_ms_per_token_step": step_ms},
        "e2e": {"value": tokens_per_step * steps / float(e2e_s[0]), "unit": unit,
                "h2d_bytes_per_step": prompts_host.numel() * 4, "d2h_bytes_per_step": out_host.numel() * 4},
        # counted by the library's launch wrapper on rank 0 inside the timed region (graph replays add the recorded
        # step's kernel count); NCCL's kernels are not this library's and are not counted
        "gpu_launches": launches,
        "clocks": clocks,
        "roofline": {"bound": "tensor", "kernel": "the tcgen05 GEMM on this run's prefill QKV / O / gate-up / down shapes "
                                                  "(gemm_bf16_2cta_kernel at config 5), timed alone after the generation (each shape from a GPU left idle for 1 s)",
                     "achieved": achieved, "peak": peaks["bf16_tflops"], "unit": "TFLOP/s",
                     "frac": achieved / peaks["bf16_tflops"],
                     "peak_source": peaks["source"] + " (burst cuBLAS bf16: the kernel is timed alone, a few launches)",
                     # DRAM bytes of the four launches together: ncu measured 0.99 x the algorithmic 2(MK + NK + MN) bytes
                     # on a 4096 x 12288 x 4096 launch of this kernel (operands read once); scaled here by algorithmic bytes
                     "traffic": 0.99 * gemm_bytes, "traffic_unit": "bytes per set of four launches, scaled from an ncu capture"},
        "roofline_prefill": {"bound": "tensor", "what": "whole prefill phase inside the step (all kernels, per GPU)",
                             "achieved": prefill_flop / (prefill_ms / steps * 1e-3) / 1e12,
                             "peak": peaks["bf16_tflops_sustained"], "unit": "TFLOP/s",
                             "frac": prefill_flop / (prefill_ms / steps * 1e-3) / 1e12 / peaks["bf16_tflops_sustained"],
                             "peak_source": peaks["source"] + " (sustained cuBLAS bf16: measured inside a long step)",
                             "flop_per_gpu": prefill_flop},
        "roofline_decode": {"bound": "hbm", "what": "one decode step (all kernels, per GPU): weights + KV cache at the mean length",
                            "achieved": decode_bytes / (step_ms * 1e-3) / 1e9, "peak": peaks["hbm_gbs"], "unit": "GB/s",
                            "frac": decode_bytes / (step_ms * 1e-3) / 1e9 / peaks["hbm_gbs"],
                            "peak_source": peaks["source"] + " (copy bandwidth)", "bytes_per_gpu": decode_bytes},
        "ids_crc32": {"all": ids_crc, "first_token": first_crc},
    }
    if parity is not None:
        line["parity_check"] = parity
    if not args.no_cpu_baseline and world == 1:
        v, desc, threads = cpu_generation_rate(cfg_kwargs, **CPU_SAMPLE[args.config])
        line["cpu_baseline"] = {"value": v, "unit": unit, "cores": threads, "kind": "port", "sample": desc}
    emit(line)
    if world > 1:
        dist.barrier()
        dist.destroy_process_group()
    if parity is not None and not parity["ok"]:
        raise SystemExit(f"parity check failed: {parity}")


# ------------------------------------------------------------------------------------------------ the hybrid decoders
# Layer sizes of real models: every layer has the feed-forward of the Qwen3 it is compared with (same width, layers, heads,
# feed-forward and vocabulary).  Fiferax layers cycle through delta, parallel, delta, mingru; Molitar's through latent
# attention and full attention.
HYBRID_SIZES = {"1k": dict(width=1024, layers=24, ff=3072, heads=16, kv_heads=8, vocab=32768,
                           latent=dict(dim=64, rot_dim=32, vdim=64, q_rank=512, kv_rank=256)),
                "4k": dict(width=4096, layers=8, ff=12288, heads=32, kv_heads=8, vocab=32768,
                           latent=dict(dim=128, rot_dim=64, vdim=128, q_rank=1536, kv_rank=512))}
FIFERAX_WINDOW, HYBRID_NEW = 1024, 128
HYBRID_WORKLOADS = [(16, 2048), (1, 2048)]


def fiferax_config_of(size):
    z = HYBRID_SIZES[size]
    W, H = z["width"], z["heads"]
    mlp = {"kind": "dense", "ff": z["ff"]}
    delta = {"type": "general_delta", "mixer": {"heads": W // 64, "dim": 64}, "mlp": mlp}
    par = {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": H, "kv_heads": z["kv_heads"], "dim": 128, "vdim": 128, "mask": {"size": FIFERAX_WINDOW},
                 "rot": {"dims": 128, "base": 1e6}, "scale": 128 ** -0.5},
        "right": {"heads": W // 128, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-1 - 9.0 * i / (W // 128)) for i in range(W // 128)]},
        "left_scale": 1.0, "right_scale": 1.0}}
    gru = {"type": "mingru", "mixer": {"width": W}, "mlp": mlp}
    return {"architecture": "Fiferax", "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5}, "vocab": z["vocab"], "width": W,
            "layers": [[delta, par, delta, gru][i % 4] for i in range(z["layers"])]}


def kernel_rows(peaks):
    """A table of kernels and the function that adds a row: achieved rate (bytes or FLOPs per launch over its time) and its
    fraction of the measured peak."""
    rows = []

    def row(kernel, ms, bound, amount, like=None):
        peak = peaks["hbm_gbs"] if bound == "hbm" else peaks["bf16_tflops"]
        ach = amount / ms / (1e6 if bound == "hbm" else 1e9)
        rows.append({"kernel": kernel, "us": ms * 1e3, "bound": bound, "achieved": ach, "unit": "GB/s" if bound == "hbm" else "TFLOP/s",
                     "frac": ach / peak, **({"like": like} if like else {})})

    return rows, row


def fiferax_kernels(size, peaks, timed, graph_timed):
    """The new design's kernels and the like ones of Qwen3, each alone at this size: (rows of the table)."""
    import torch
    from teenygrad_b200 import ops
    from teenygrad_b200._lib import lib
    z = HYBRID_SIZES[size]
    W, H, G, win = z["width"], z["heads"], z["kv_heads"], FIFERAX_WINDOW
    B, S = HYBRID_WORKLOADS[0]
    T, H64, H128, D = B * S, W // 64, W // 128, 128
    g = torch.Generator(device="cuda").manual_seed(3)
    rnd = lambda *s: torch.randn(*s, generator=g, device="cuda")  # noqa: E731
    bf = lambda *s: rnd(*s).bfloat16()  # noqa: E731
    rows, row = kernel_rows(peaks)
    whole = ops.seq_table([(b, 0, b * S, S) for b in range(B)])
    proj = bf(T, 6 * W)
    wz = bf(T, W)
    bias = rnd(W)
    offs = (0, W, 2 * W, 3 * W)
    st64 = torch.zeros(B, H64, 64, 64, device="cuda")
    o32, o16 = rnd(T, W), bf(T, W)
    row("state scan, delta rule (prefill)", timed(lambda: ops.state_scan_delta(proj, offs, wz, bias, bias, 0.6, 1e-6, st64, whole, S, out=o32)), "hbm",
        T * W * (5 * 2 + 4), "attention, prefill")
    st128 = torch.zeros(B, H128, 128, 128, device="cuda")
    decay = torch.full((H128,), 0.99, device="cuda")
    row("state scan, scalar decay (prefill)", timed(lambda: ops.state_scan_decay(proj, offs[:3], decay, st128, whole, S, out=o32)), "hbm",
        T * W * (3 * 2 + 4), "attention, prefill")
    w32 = torch.ones(W, device="cuda")
    row("gated norm per head", timed(lambda: ops.gated_rms_norm(o32, wz, w32, 64, 1e-5, out=o16)), "hbm", T * W * 8, "residual add + norm, bf16")
    row("gated norm over all heads", timed(lambda: ops.gated_rms_norm(o32, wz, w32, W, 1e-5, out=o16)), "hbm", T * W * 8, "residual add + norm, bf16")
    gs = torch.zeros(B, W, device="cuda")
    row("minimal GRU scan (prefill)", timed(lambda: ops.min_gru(proj, offs[:3], bias, bias, gs, whole, S, out=o16)), "hbm", T * W * 8,
        "residual add + norm, bf16")
    q, k = proj[:, :H * D].view(T, H, D), proj[:, H * D:(H + G) * D].view(T, G, D)
    inv, nw = torch.rand(D // 2, device="cuda", generator=g), torch.ones(D, device="cuda")
    kc, oa = k.contiguous(), bf(T, H, D)
    row("head norm + rotary, f32 angles", timed(lambda: ops.head_norm_rope(q, k, nw, nw, inv, D, 1e-5, whole, S, out=kc)), "hbm",
        2 * 2 * T * (H + G) * D, "head norm + rotary + cache, bf16 tables")
    kr, vr = (torch.zeros(B, G, win, D, dtype=torch.bfloat16, device="cuda") for _ in range(2))
    seen = sum(min(i + 1, win) for i in range(S))
    row("windowed attention (prefill) + ring append", timed(lambda: ops.window_attention(q, kc, k, kr, vr, win, D ** -0.5, whole, S,
                                                                                         uniform_fresh=True, out=oa)),
        "tensor", 4.0 * B * H * D * seen, "attention, prefill")
    x32, delta = rnd(T, W), bf(T, W)
    row("residual add + norm, f32 residual", timed(lambda: ops.residual_rms_norm(x32, delta, w32, 1e-5)), "hbm", T * W * 12,
        "residual add + norm, bf16")
    # one token per sequence, batch 32, states / caches rotated beyond L2
    n, copies = 32, 8
    one = ops.seq_table([(b, S, b, 1) for b in range(n)])
    p1, z1, o1 = proj[:n], wz[:n], o32[:n]
    s64 = [torch.zeros(n, H64, 64, 64, device="cuda") for _ in range(copies)]
    row("state step, delta rule (decode)", graph_timed([(lambda s=s: ops.state_scan_delta(p1, offs, z1, bias, bias, 0.6, 1e-6, s, one, 1, out=o1))
                                                        for s in s64]), "hbm", 2.0 * n * H64 * 64 * 64 * 4, "attention, decode")
    del s64
    s128 = [torch.zeros(n, H128, 128, 128, device="cuda") for _ in range(copies)]
    row("state step, scalar decay (decode)", graph_timed([(lambda s=s: ops.state_scan_decay(p1, offs[:3], decay, s, one, 1, out=o1)) for s in s128]),
        "hbm", 2.0 * n * H128 * 128 * 128 * 4, "attention, decode")
    del s128
    # decode attention over full rings: min(pos + 1, window) keys
    from teenygrad_b200.ops import flash_attn_decode
    for length, name in ((win, "attention, decode (ring of the window)"), (S, "attention, decode")):
        kvs = [(bf(n, G, length, D), bf(n, G, length, D)) for _ in range(6)]
        q1 = bf(n, H, 1, D)
        o1 = torch.empty_like(q1)
        sc = torch.empty(lib.teeny_attn_decode_scratch_bytes(n, H, D, length), dtype=torch.uint8, device="cuda")
        row(name, graph_timed([(lambda kk=kk, vv=vv: flash_attn_decode(q1, kk, vv, length, D ** -0.5, out=o1, scratch=sc)) for kk, vv in kvs]),
            "hbm", 2.0 * n * G * length * D * 2, "attention, decode" if length == win else None)
        del kvs
    qwen3_kernels(z, B, S, row, timed)
    return rows


def molitar_config_of(size):
    z = HYBRID_SIZES[size]
    H, lat = z["heads"], z["latent"]
    mlp = {"kind": "dense", "ff": z["ff"]}
    latent = {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": H, **lat, "scale": (lat["dim"] + lat["rot_dim"]) ** -0.5,
        "rot": {"dims": lat["rot_dim"], "base": 1e6, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    full = {"type": "attention", "mlp": mlp, "mixer": {
        "heads": H, "kv_heads": z["kv_heads"], "dim": 128, "vdim": 128, "rot": {"dims": 64, "base": 1e6}, "scale": 128 ** -0.5,
        "softcap": 30.0, "v_mix": True}}
    return {"architecture": "Molitar", "logit_scale": 0.25, "norm": {"eps": 1e-6}, "residual_mult": 0.7, "vocab": z["vocab"],
            "width": z["width"], "layers": [[latent, full][i % 2] for i in range(z["layers"])]}


def molitar_kernels(size, peaks, timed, graph_timed):
    """The design's kernels and the like ones of Qwen3, each alone at this size."""
    import torch
    from teenygrad_b200 import ops
    z = HYBRID_SIZES[size]
    W, H, G, D, lat = z["width"], z["heads"], z["kv_heads"], 128, z["latent"]
    B, S = HYBRID_WORKLOADS[0]
    T = B * S
    g = torch.Generator(device="cuda").manual_seed(3)
    rnd = lambda *s: torch.randn(*s, generator=g, device="cuda")  # noqa: E731
    bf = lambda *s: rnd(*s).bfloat16()  # noqa: E731
    rows, row = kernel_rows(peaks)
    table = lambda entries: (ops.seq_table(entries), ops.seq_table(entries, "cpu"))  # noqa: E731
    whole = table([(b, 0, b * S, S) for b in range(B)])
    causal = lambda d: 2.0 * B * H * d * S * (S + 1) / 2  # noqa: E731  (FLOPs of one product per visible pair)
    # ---- prompts
    sink, inv = rnd(H), torch.rand(D // 2, device="cuda", generator=g)
    q, out, gate = bf(T, H, D), bf(T, H, D), bf(T, H * D)
    kc, vc = bf(B, G, S, D), bf(B, G, S, D)
    row("full attention (cap, sink) + output gate, prefill", timed(lambda: ops.cached_attention(q, kc, vc, D ** -0.5, whole, softcap=30.0, sink=sink,
                                                                                             gate=gate, out=out)),
        "tensor", causal(2 * D), "attention, prefill")
    proj, first, lam = bf(T, (H + 2 * G) * D), bf(T, G * D), torch.full((1,), 0.5, device="cuda")
    qp, kp, vp = (proj[:, a * D:b * D].view(T, -1, D) for a, b in ((0, H), (H, H + G), (H + G, H + 2 * G)))
    row("rotary + value mixing + cache", timed(lambda: ops.rope_cache(qp, kp, vp, kc, vc, inv, 64, whole[0], S, v_first=first, mix=lam)), "hbm",
        2.0 * T * D * (2 * H + 5 * G), "head norm + rotary + cache, bf16 tables")
    del proj, first
    KD, V, R, RD, QR = lat["dim"] + lat["rot_dim"], lat["vdim"], lat["kv_rank"], lat["rot_dim"], lat["q_rank"]
    ql, ol = bf(T, H, KD), bf(T, H, V)
    kl, vl = bf(B, H, S, KD), bf(B, H, S, V)
    row("latent attention, expanded, prefill", timed(lambda: ops.cached_attention(ql, kl, vl, KD ** -0.5, whole, out=ol)), "tensor", causal(KD + V),
        "attention, prefill")
    del kl, vl, ql, ol, q, out, gate
    down, cache, latents = bf(T, QR + R + RD), bf(B, S, R + RD), bf(T, R + RD)
    qw, cw = torch.ones(QR, device="cuda"), torch.ones(R, device="cuda")
    row("latent norms + rotary + cache", timed(lambda: ops.latent_prepare(down, (0, QR, QR + R), QR, R, qw, cw, inv, 1e-6, cache, whole[0], S,
                                                                       latents=latents)), "hbm",
        2.0 * T * (2 * QR + 3 * (R + RD)), "head norm + rotary + cache, bf16 tables")
    del down, cache, latents
    x32, delta, w32 = rnd(T, W), bf(T, W), torch.ones(W, device="cuda")
    row("norm + residual add + norm, f32 residual", timed(lambda: ops.residual_rms_norm(x32, delta, w32, 1e-6, w32, 0.7)), "hbm", T * W * 12,
        "residual add + norm, bf16")
    del x32, delta
    # ---- one token per sequence, weights and caches rotated beyond L2
    n, copies = B, 6
    one = table([(b, S - 1, b, 1) for b in range(n)])
    q1, o1, g1 = bf(n, H, D), bf(n, H, D), bf(n, H * D)
    from teenygrad_b200._lib import lib
    scratch = (torch.empty(lib.teeny_attn_decode_scratch_bytes(n, H, 128, S), dtype=torch.uint8, device="cuda"),
               torch.zeros(n * G, dtype=torch.int32, device="cuda"))
    kvs = [(bf(n, G, S, D), bf(n, G, S, D)) for _ in range(copies)]
    row("full attention (cap, sink, gate), decode", graph_timed([(lambda k=k, v=v: ops.cached_attention(
        q1, k, v, D ** -0.5, one, softcap=30.0, sink=sink, gate=g1, out=o1, scratch=scratch)) for k, v in kvs]), "hbm", 2.0 * n * G * S * D * 2,
        "attention, decode")
    del kvs
    ql, ol = bf(n, H, R + RD), bf(n, H, R)
    part = torch.empty(lib.teeny_latent_attention_scratch_bytes(R), dtype=torch.uint8, device="cuda")
    for length, name in ((S, ""), (4 * S, f", context {4 * S}")):
        at = ops.seq_table([(b, length - 1, b, 1) for b in range(n)])
        caches = [bf(n, length, R + RD) for _ in range(copies + 2 if length == S else 3)]
        row("latent attention, absorbed, decode" + name, graph_timed([(lambda c=c, at=at: ops.latent_attention(ql, c, R, KD ** -0.5, at, 1, out=ol, scratch=part))
                                                                       for c in caches]), "hbm", 2.0 * n * length * (R + RD), "attention, decode" + name)
        del caches
    qh, vo = bf(n, H, KD), bf(n, H, V)
    many = max(8, (300 << 20) // (2 * H * R * lat["dim"]))
    ws = [bf(H, R, lat["dim"]) for _ in range(many)]
    row("queries into the latent space + rotary, decode", graph_timed([(lambda w=w: ops.head_linear(
        qh[:, :, RD:], w, RD, -RD, inv, 1.0, one[0], out=ql)) for w in ws]), "hbm", 2.0 * H * R * lat["dim"], "matrix product, decode")
    ws = [bf(H, V, R) for _ in range(many)]
    row("values out of the latent space, decode", graph_timed([(lambda w=w: ops.head_linear(ol, w, out=vo)) for w in ws]), "hbm", 2.0 * H * R * V,
        "matrix product, decode")
    ws = [bf(H * V, R) for _ in range(many)]
    x1 = bf(n, R)
    row("matrix product, decode", graph_timed([(lambda w=w: ops.linear_forward(x1, w)) for w in ws]), "hbm", 2.0 * H * R * V)
    del ws
    qwen3_kernels(z, B, S, row, timed)
    from teenygrad_b200.ops import flash_attn_decode
    qd = bf(n, H, 1, D)
    od = torch.empty_like(qd)
    for length, name in ((S, ""), (4 * S, f", context {4 * S}")):
        kvs = [(bf(n, G, length, D), bf(n, G, length, D)) for _ in range(copies if length == S else 2)]
        sc = torch.empty(lib.teeny_attn_decode_scratch_bytes(n, H, D, length), dtype=torch.uint8, device="cuda")
        row("attention, decode" + name, graph_timed([(lambda k=k, v=v, length=length: flash_attn_decode(qd, k, v, length, D ** -0.5, out=od, scratch=sc))
                                                     for k, v in kvs]), "hbm", 2.0 * n * G * length * D * 2)
        del kvs
    return rows


def qwen3_kernels(z, B, S, row, timed):
    """The like kernels of the Qwen3 runner over prompts."""
    import torch
    from teenygrad_b200 import ops
    from teenygrad_b200.ops import flash_attn_fwd
    W, H, G, D, T = z["width"], z["heads"], z["kv_heads"], 128, B * S
    bf = lambda *s: torch.randn(*s, device="cuda").bfloat16()  # noqa: E731
    qa, ka = bf(B, H, S, D), bf(B, G, S, D)
    row("attention, prefill", timed(lambda: flash_attn_fwd(qa, ka, ka, D ** -0.5, causal=True)), "tensor", 0.5 * 4 * B * H * S * S * D)
    delta, xr, w16 = bf(T, W), bf(T, W), torch.ones(W, dtype=torch.bfloat16, device="cuda")
    row("residual add + norm, bf16", timed(lambda: ops.add_rms_norm(delta, xr, w16, 1e-5)), "hbm", T * W * 8)
    cos, sin = ops.rope_table(torch.rand(D // 2, device="cuda"), S)
    qkv, n16 = bf(T, (H + 2 * G) * D), torch.ones(D, dtype=torch.bfloat16, device="cuda")
    kk, vv = (torch.zeros(B, G, S, D, dtype=torch.bfloat16, device="cuda") for _ in range(2))
    row("head norm + rotary + cache, bf16 tables", timed(lambda: ops.qk_norm_rope_kv(qkv, n16, n16, cos, sin, kk, vv, S, H, G, 0, 1e-6)), "hbm",
        2.0 * T * D * (2 * H + 4 * G))


def hybrid_bench(args):
    import torch
    from teenygrad_b200 import fiferax, molitar, qwen3
    from teenygrad_b200._lib import lib
    name = args.model
    if args.gpus != 1 or args.impl != "ours":
        raise SystemExit(f"--model {name} runs on one GPU")
    torch.cuda.set_device(0)
    peaks, z, NEW = measured_peaks(), HYBRID_SIZES[args.size], HYBRID_NEW
    if name == "fiferax":
        rank = z["width"] // 32
        cfg, kernel_table = fiferax_config_of(args.size), fiferax_kernels
        shapes, tensors, module = fiferax.tensor_shapes(cfg, rank), fiferax.RandomTensors(cfg, 7, "cuda", rank), fiferax
        layers = f"delta, parallel, delta, mingru), window {FIFERAX_WINDOW}"
    else:
        cfg, kernel_table = molitar_config_of(args.size), molitar_kernels
        shapes, tensors, module = molitar.tensor_shapes(cfg), molitar.RandomTensors(cfg, 7, "cuda"), molitar
        layers = f"latent attention, full attention), latents {z['latent']}"
    warm = max(args.warmup, 3)
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def timed(fn, steps=5):
        for _ in range(3):
            fn()
        total = 0.0
        for _ in range(steps):
            flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            total += a.elapsed_time(b)
        return total / steps

    def graph_timed(fns, reps=5):
        st = torch.cuda.Stream()
        with torch.cuda.stream(st):
            for f in fns:
                f()
            torch.cuda.synchronize()
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph, stream=st):
                for f in fns:
                    f()
            for _ in range(3):
                graph.replay()
            torch.cuda.synchronize()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            for _ in range(reps):
                graph.replay()
            b.record()
            torch.cuda.synchronize()
        return a.elapsed_time(b) / reps / len(fns)

    def phases(prefill, decode, steps):
        for _ in range(warm):
            prefill()
            for _ in range(3):
                decode()
        ev = [[torch.cuda.Event(enable_timing=True) for _ in range(3)] for _ in range(steps)]
        torch.cuda.synchronize()
        for e in ev:
            e[0].record()
            prefill()
            e[1].record()
            for _ in range(NEW - 1):
                decode()
            e[2].record()
        torch.cuda.synchronize()
        return [sum(e[i].elapsed_time(e[i + 1]) for e in ev) / steps for i in range(2)]

    def matmul_params(model):
        if model == "qwen3":
            return z["layers"] * (z["width"] * (2 * z["heads"] + 2 * z["kv_heads"]) * 128 + 3 * z["width"] * z["ff"]) + z["vocab"] * z["width"]
        return sum(s[0] * s[1] for n, s in shapes.items() if len(s) == 2 and (n != "embed" or "head" not in shapes))

    sampler = ClockSampler(0)
    sampler.start()
    results, launches, e2e = [], 0, None
    for B, S in HYBRID_WORKLOADS:
        g = torch.Generator().manual_seed(6)
        host = torch.randint(0, z["vocab"], (B, S), generator=g, dtype=torch.int32).pin_memory()
        dev = host.cuda()
        entry = {"batch": B, "prefill": S, "new_tokens": NEW}
        for model in (name, "qwen3"):
            if model == name:
                r = module.build(cfg, tensors, max_batch=B, max_len=S + NEW, max_tokens=B * S, max_new_tokens=NEW)
                seqs = [r.open() for _ in range(B)]

                def prefill():
                    for s in seqs:
                        s.pos = 0
                    r.prefill(dev, seqs)
            else:
                r = qwen3.Qwen3Runner(qwen3.Qwen3Config(z["layers"], z["width"], z["heads"], z["kv_heads"], 128, z["ff"], z["vocab"]), max_batch=B,
                                      max_len=S + NEW, max_tokens=B * S, max_new_tokens=NEW)
                qwen3.load_random_weights(r, 7)

                def prefill():
                    r.prefill(dev)
            lib.teeny_launch_count(1)
            pre, dec = phases(prefill, lambda: r.decode_step(graph=True), args.steps)
            if model == name:
                launches += int(lib.teeny_launch_count(1))
            entry[model] = {"prefill_ms": pre, "decode_ms_per_step": dec / (NEW - 1), "prefill_tok_s": B * S / pre * 1e3,
                            "decode_tok_s": B * (NEW - 1) / dec * 1e3, "tok_s": B * (S + NEW) / (pre + dec) * 1e3,
                            "matmul_params": matmul_params(model),
                            "prefill_matmul_tflops": 2.0 * matmul_params(model) * B * S / pre / 1e9,
                            "decode_weight_gbs": 2.0 * matmul_params(model) / (dec / (NEW - 1)) / 1e6}
            if model == name and e2e is None:
                for s in seqs:
                    r.close(s)
                out = torch.empty(B, NEW, dtype=torch.int32).pin_memory()

                def once():
                    out.copy_(r.generate(host.to("cuda", non_blocking=True), NEW), non_blocking=True)
                    torch.cuda.current_stream().synchronize()
                once()
                t0 = time.perf_counter()
                for _ in range(args.steps):
                    once()
                e2e = {"value": B * (S + NEW) * args.steps / (time.perf_counter() - t0), "unit": "tok/s", "h2d_bytes_per_step": host.numel() * 4,
                       "d2h_bytes_per_step": out.numel() * 4}
            if r.device_error():
                raise SystemExit("device error word set")
            del r
            torch.cuda.empty_cache()
        results.append(entry)
    clocks = sampler.stop()
    kernels = kernel_table(args.size, peaks, timed, graph_timed)
    first = results[0]
    emit({"metric": f"{name}_tokens_per_s", "value": first[name]["tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": args.steps,
          "warmup": args.warmup, "warmup_run": warm,
          "ms_per_step": first[name]["prefill_ms"] + first[name]["decode_ms_per_step"] * (NEW - 1), "higher_is_better": True,
          "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
          "config": {"workload": f"{name.capitalize()} {args.size}: width {z['width']}, {z['layers']} layers ({layers}, "
                                 f"feed-forward {z['ff']}, vocabulary {z['vocab']}, random weights; beside a Qwen3 of the same "
                                 "width, layers, heads, feed-forward and vocabulary", "parallelism": "1 GPU",
                     "l2": "inputs larger than L2; kernels alone: L2 flushed before every timed launch, one-token kernels replayed from a graph "
                           "over state copies larger than L2"},
          "workloads": results, "kernels": kernels, "e2e": e2e, "gpu_launches": launches, "clocks": clocks})


def main():
    args = parse_args()
    # Keep stdout to the one JSON line: libraries write there at the file-descriptor level (NCCL prints its version
    # banner to fd 1 at NCCL_DEBUG=VERSION and WARN), so fd 1 is pointed at stderr for the whole run and the line goes
    # to a private duplicate of the original stdout.
    global _JSON_OUT
    sys.stdout.flush()
    _JSON_OUT = os.fdopen(os.dup(1), "w")
    os.dup2(2, 1)
    if args.model != "qwen3":
        hybrid_bench(args)
    elif args.impl == "reference":
        reference_arm(args)
    elif args.config in (4, 5):
        generation_config(args)
    else:
        kernel_config(args)


if __name__ == "__main__":
    main()
