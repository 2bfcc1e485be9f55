"""Headline benchmark: training throughput (tokens/s) of a GPT-J-6B-shape decoder, bf16 compute with fp32 master
weights and fp32 Adam state, sequence length 2048, 16 micro-batches of 1 sequence per data-parallel replica and step,
tensor parallel x data parallel with the optimizer state sharded over the data-parallel group (TP4 x DP2 on 8 GPUs).

    python bench.py [--gpus N] [--steps K] [--warmup W] [--impl ours|reference] [--model gptj_6b|gpt2_small|llama2_7b]

With N > 1 it is launched by `python -m torch.distributed.run --nproc-per-node N ... bench.py --gpus N ...` (one rank per
GPU). Rank 0 prints one JSON line. `value` is timed on the device with CUDA events around K steps whose inputs are
already resident; `e2e` is timed around the public `DecoderTrainer.step` call, which copies each step's tokens from
pinned host memory and reads the losses back.
"""
import argparse
import json
import os
import subprocess
import sys
import threading
import time

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

METRIC = "train tokens/s GPT-J-6B shape TPxDP (bf16, fp32 Adam, seq 2048, 16 micro-batches of 1)"


def layout_for(n_gpus: int):
    tp = min(n_gpus, 4)
    return tp, n_gpus // tp


class ClockSampler:
    """Polls nvidia-smi while the timed region runs (SM clock and throttle reasons of this rank's GPU)."""

    FIELDS = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
              "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
              "clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int):
        self.index, self.samples, self._stop, self._thread = index, [], threading.Event(), None

    def _loop(self):
        while not self._stop.is_set():
            try:
                out = subprocess.run(["nvidia-smi", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits",
                                      "-i", str(self.index)], capture_output=True, text=True, timeout=5).stdout
                parts = [p.strip() for p in out.strip().split(",")]
                if len(parts) >= 7:
                    self.samples.append(parts)
            except Exception:
                pass
            self._stop.wait(0.2)

    def __enter__(self):
        self._thread = threading.Thread(target=self._loop, daemon=True)
        self._thread.start()
        return self

    def __exit__(self, *exc):
        self._stop.set()
        self._thread.join(timeout=6)

    def summary(self):
        if not self.samples:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": []}
        sm = sorted(float(s[0]) for s in self.samples if s[0].replace(".", "").isdigit())
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(s[3 + i].lower().startswith("active") for s in self.samples)]
        mx = [float(s[1]) for s in self.samples if s[1].replace(".", "").isdigit()]
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": reasons, "samples": len(self.samples)}


def run_reference(args):
    """Runs the unmodified reference from `baseline/_ref` if it can be imported. It needs Graphcore's Poplar SDK
    (`popxl`, `popart`) and an IPU, so on this platform the import fails and the arm reports itself unavailable."""
    ref = os.path.join(os.path.dirname(os.path.abspath(__file__)), "baseline", "_ref")
    why = None
    if not os.path.isdir(os.path.join(ref, "popxl_addons")):
        why = "baseline/_ref/popxl_addons is not installed"
    else:
        sys.path.insert(0, ref)
        try:
            import popxl_addons  # noqa: F401
        except Exception as e:  # ModuleNotFoundError: No module named 'popxl'
            why = (f"`import popxl_addons` from baseline/_ref fails with {type(e).__name__}: {e} "
                   "(the reference is a layer on Graphcore's Poplar SDK, which exists only for IPU systems)")
    if why is None:
        why = "the reference imported, but it can only execute on Graphcore IPU hardware (popxl.Session needs an IPU)"
    if int(os.environ.get("RANK", "0")) == 0:  # one line per job, also when launched with one process per GPU
        print(json.dumps({"impl": "reference", "unavailable": why}))
    return 0


PIPELINE_METRIC = "train tokens/s Llama-2-7B shape PPxDP (bf16, fp32 Adam, seq 2048, 32 micro-batches of 1)"
DECODE_METRIC = "int4 decode tokens/s GPT-J-6B shape, TP over all GPUs (batch 16, prompt 512, 128 new tokens, greedy)"


def _shrink(cfg, k: int):
    """One rank's share of a k-way tensor-parallel layout as a stand-alone model (diagnostics only)."""
    cfg.heads //= k
    cfg.ffn //= k
    cfg.vocab_size = (cfg.vocab_size + k - 1) // k


def _shutdown(dist):
    """Leave without tearing the NCCL communicators down: destroying them while captured CUDA graphs that contain
    their kernels are still alive has been seen to block for minutes."""
    if dist is not None:
        dist.barrier()
    sys.stdout.flush()
    sys.stderr.flush()
    if dist is not None:
        os._exit(0)


def run_decode(args, standalone: bool = True):
    """Int4 group-quantised greedy generation: weights N(0, 0.02) quantised in groups of 64 along the input dimension
    with fp16 scale and bias, bf16 activations and KV cache, tensor parallel over all GPUs. One step = one whole
    `generate` call (prefill of the prompts + `new_tokens - 1` single-token steps). With `standalone=False` the record
    is returned (rank 0; None elsewhere) instead of printed, and the process is not ended."""
    import numpy as np
    import torch

    from popxl_addons_b200.models.decoder import DecoderConfig

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if world != args.gpus and world == 1 and args.gpus > 1:
        raise SystemExit("launch with torch.distributed.run --nproc-per-node N for --gpus N > 1")
    torch.cuda.set_device(local_rank)
    cfg = getattr(DecoderConfig, args.model)(tp=args.gpus, dp=1)
    if args.layers:
        cfg.layers = args.layers
    if args.emulate_tp:
        _shrink(cfg, args.emulate_tp)
    W, K = max(args.warmup, 3), args.steps
    B, P, N = args.batch, args.prompt_len, args.new_tokens
    t0 = time.perf_counter()
    if args.impl == "torch":
        sys.path.insert(0, os.path.join(os.path.dirname(os.path.abspath(__file__)), "baseline"))
        from torch_generator import TorchGenerator

        gen = TorchGenerator(cfg, B, P, N, group_size=64, cache_dense=args.torch_dense,
                             cuda_graph=not args.no_cuda_graphs)
        launches_of = lambda: 0  # noqa: E731
        kernels_of = lambda: {}  # noqa: E731
    else:
        from popxl_addons_b200.models.generator import DecoderGenerator
        from popxl_addons_b200.ops import native

        gen = DecoderGenerator(cfg, B, P, N, group_size=64, device="cuda", seed=0, cuda_graphs=not args.no_cuda_graphs)
        launches_of = lambda: native.LAUNCHES["count"]  # noqa: E731
        kernels_of = lambda: native.LAUNCHES["by_kernel"]  # noqa: E731
    setup_s = time.perf_counter() - t0
    dist = torch.distributed if world > 1 else None

    def barrier():
        if dist is not None:
            dist.barrier()
        torch.cuda.synchronize()

    rs = np.random.RandomState(0)
    prompts = [torch.from_numpy(rs.randint(0, cfg.vocab_size, (B, P)).astype(np.int32)).pin_memory() for _ in range(W + K)]
    for i in range(W):
        out = gen.generate(prompts[i])
    launches0 = launches_of()
    dev_ms = prefill_ms = decode_ms = 0.0
    with ClockSampler(local_rank) as clocks:
        barrier()
        t1 = time.perf_counter()
        for i in range(K):
            out = gen.generate(prompts[W + i])  # pinned prompt -> device, program, tokens -> host
            prefill_ms += gen.prefill_ms()
            decode_ms += gen.decode_ms()
        barrier()
        e2e_s = time.perf_counter() - t1
    dev_ms = prefill_ms + decode_ms  # CUDA events recorded by the program around its two phases
    launches = launches_of() - launches0
    times = torch.tensor([dev_ms, e2e_s * 1e3, prefill_ms, decode_ms], dtype=torch.float64, device="cuda")
    if dist is not None:
        dist.all_reduce(times, op=dist.ReduceOp.MAX)
    dev_ms, e2e_ms, prefill_ms, decode_ms = (float(t) for t in times)
    if args.impl != "torch":
        native.check_gemm_errors()
    line = None
    if rank == 0:
        toks = B * N * K
        line = {
            "impl": args.impl, "metric": DECODE_METRIC, "value": toks / (dev_ms / 1e3), "unit": "tokens/s",
            "n_gpus": args.gpus, "steps": K, "warmup": W, "ms_per_step": dev_ms / K, "higher_is_better": True,
            "scaling": "strong", "vs_baseline": None, "dtype": "bf16 activations and KV cache, int4 weights (fp16 scales)",
            "data": "synthetic (uniform random prompt ids, random-init N(0,0.02) weights quantised to int4)",
            "config": {"model": f"{args.model} ({cfg.layers} layers, hidden {cfg.hidden}, {cfg.heads} heads x "
                                f"{cfg.head_dim}, ffn {cfg.ffn}, vocab {cfg.vocab_size})",
                       "global_batch": B, "seq_len": P + N, "prompt_len": P, "new_tokens": N,
                       "parallelism": f"tp{args.gpus}", "group_size": 64,
                       "cuda_graphs": not args.no_cuda_graphs,
                       "torch_weights": ("bf16 copy cached" if args.torch_dense else "int4, de-quantised per call")
                       if args.impl == "torch" else None,
                       "l2": "every decoding step streams all int4 weights and the KV cache (several GB in total), "
                             "beyond the 126 MB L2; no flush needed",
                       "headline": (not args.layers and not args.emulate_tp and args.model == "gptj_6b"
                                    and (B, P, N) == (16, 512, 128)),
                       "emulate_tp": args.emulate_tp or None},
            "clocks": clocks.summary(),
            "e2e": {"value": toks / (e2e_ms / 1e3), "unit": "tokens/s", "ms_per_step": e2e_ms / K,
                    "h2d_bytes_per_step": B * P * 4, "d2h_bytes_per_step": B * N * 4},
            "gpu_launches": int(launches), "kernels": kernels_of(),
            "prefill_ms": prefill_ms / K, "decode_ms": decode_ms / K,
            "decode_only_tokens_per_s": B * (N - 1) * K / (decode_ms / 1e3),
            "ms_per_decode_step": decode_ms / K / (N - 1),
            "sample_tokens": [int(t) for t in np.asarray(out)[0, :8]], "setup_seconds": setup_s,
        }
    del gen
    _free_device_memory()
    if not standalone:
        return line
    if rank == 0:
        print(json.dumps(line))
    _shutdown(dist)
    return 0


SERVING_METRIC = "serving tokens/s {} layers (bf16, batch 16, prompt 512, 64 new tokens, greedy)"

# name: width, feed-forward, recurrent width, query heads, key / value heads (of 128 features, or two maps of 64 with values
# of 128)
SERVING_SIZES = {"w2048": (2048, 5632, 2048, 16, 4), "w4096": (4096, 11008, 4096, 32, 8), "w8192": (8192, 22016, 8192, 64, 8)}


def _dunelix_serving(C, F, R, H, G, vocab, layers, chunk):
    """Dunelix of four layers, one letter each: r recurrent (minGRU), a differential attention."""
    from popxl_addons_b200.models.dunelix import Dunelix, DunelixConfig

    gru = {"type": "mingru", "mixer": {"width": R}, "mlp": {"ff": F, "kind": "dense"}}
    att = {"type": "attention", "mlp": {"ff": F, "kind": "dense"},
           "mixer": {"heads": H, "kv_heads": G, "dim": 64, "vdim": 128, "diff": 0.5, "scale": 0.125, "mask": {"size": chunk},
                     "rot": {"base": 500000.0, "dims": 64,
                             "scaling": {"factor": 16.0, "low": 1.0, "high": 4.0, "original": 4096}}}}
    return Dunelix(DunelixConfig.from_dict({"vocab": vocab, "width": C, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
                                            "layers": [{"r": gru, "a": att}[k] for k in layers]}))


def _zirunex_serving(C, F, H, G, vocab, window):
    from popxl_addons_b200.models.zirunex import Zirunex, ZirunexConfig

    layer = {"type": "attention", "mlp": {"ff": F, "kind": "dense", "limit": 7.0},
             "mixer": {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                       "mask": {"size": window, "keep_first": 4}}}
    return Zirunex(ZirunexConfig.from_dict({"vocab": vocab, "width": C, "norm": {"eps": 1e-6}, "embedding": {"scale": 8.0},
                                            "layers": [layer] * 4}))


def run_serving(args):
    """Prefill and decoding of a sequence model at sizes that resemble a real model's layers (four layers, random weights),
    beside the closest other model with as many parameters per layer. `dunelix`: three minGRU and one differential attention
    with chunks of 8192, beside the GPT-J-style `DecoderGenerator` (int4 weights). `zirunex`: four layers of attention with
    windows of 256, beside Dunelix with four attention layers and chunks of 256. One step = one `generate` call: 16 prompts of
    512 tokens and 64 new tokens. `value` is the total of prompt and new tokens of the middle size per second of device time."""
    import numpy as np
    import torch

    from popxl_addons_b200.models.decoder import DecoderConfig
    from popxl_addons_b200.models.generator import DecoderGenerator
    from popxl_addons_b200.models.sequence_generator import SequenceGenerator
    from popxl_addons_b200.ops import native

    torch.cuda.set_device(0)
    W, K, B, P, N, vocab = max(args.warmup, 3), args.steps, args.batch, args.prompt_len, args.new_tokens, 32000
    if N == 128:
        N = 64
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    path = os.path.join(os.path.dirname(os.path.abspath(__file__)), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        peaks.update(json.load(open(path)))
    rs = np.random.RandomState(0)
    prompts = [rs.randint(0, vocab, (B, P)).astype(np.int32) for _ in range(W + K)]
    records, launches_total = [], 0

    def measure(gen, as_lists):
        nonlocal launches_total
        data = [p.tolist() for p in prompts] if as_lists else prompts
        call = (lambda p: gen.generate(p, N)) if as_lists else gen.generate
        for i in range(W):
            call(data[i])
        before = native.LAUNCHES["count"]
        pre = dec = 0.0
        with ClockSampler(0) as clocks:
            torch.cuda.synchronize()
            t = time.perf_counter()
            for i in range(K):
                call(data[W + i])
                pre, dec = pre + gen.prefill_ms(), dec + gen.decode_ms()
            torch.cuda.synchronize()
            wall = (time.perf_counter() - t) * 1e3
        launches_total += native.LAUNCHES["count"] - before
        return dict(prefill_ms=pre / K, ms_per_decode_step=dec / K / (N - 1), e2e_ms=wall / K, clocks=clocks.summary())

    def serve(model):
        gen = SequenceGenerator(model, batch=B, max_seq=P + N, max_portion=P, max_new_tokens=N, device="cuda",
                                cuda_graphs=not args.no_cuda_graphs)
        gen.load(model.random_weights(0, gen.session.device))
        return measure(gen, True)

    design, window = {"dunelix": "Dunelix", "zirunex": "Zirunex"}[args.mode], 256
    for name, (C, F, R, H, G) in SERVING_SIZES.items():
        if args.model != "gptj_6b" and args.model != name:
            continue
        if design == "Dunelix":
            model = _dunelix_serving(C, F, R, H, G, vocab, "rrar", 8192)
            # two maps, half of the square; one attention layer
            att_flops, kv = 4 * (64 + 128) * P * P / 2 * H, B * (P + N / 2) * G * 256 * 2
        else:
            model = _zirunex_serving(C, F, H, G, vocab, window)
            pairs, seen = window * P - window * (window - 1) / 2, min(window + 4, P)
            att_flops, kv = 4 * 2 * (128 + 128) * pairs * H, 4 * B * seen * G * 256 * 2
        body = model.cfg.param_count() - 2 * vocab * C
        ours = serve(model)
        _free_device_memory()
        if design == "Dunelix":
            like_name, ffn = "gptj_int4", max(128, int((body / 4 - 4 * C * C) / (2 * C)) // 128 * 128)
            jcfg = DecoderConfig(family="gptj", layers=4, hidden=C, heads=C // 128, head_dim=128, rotary_dim=64, ffn=ffn,
                                 vocab_size=vocab, seq_len=P + N)
            gen = DecoderGenerator(jcfg, B, P, N, group_size=64, device="cuda", seed=0, cuda_graphs=not args.no_cuda_graphs)
            like, like_body = measure(gen, False), body
            like_bytes = (body + vocab * C) * (0.5 + 4 / 64) + B * (P + N / 2) * 2 * C * 2
            like_att = 2 * P * P * C
            del gen
        else:
            like_name = "dunelix"
            ffn = F + (body // 4 - C * (2 * (H + G) * 64 + (G + H) * 128 + 3 * F)) // (3 * C) // 64 * 64
            other = _dunelix_serving(C, ffn, R, H, G, vocab, "aaaa", window)
            like, like_body = serve(other), other.cfg.param_count() - 2 * vocab * C
            # decoding sees half a chunk on average, prompts half of every chunk's square
            like_bytes = (like_body + vocab * C) * 2 + 4 * B * (window / 2) * G * 256 * 2
            like_att = 4 * 4 * (64 + 128) * P * window / 2 * H
        _free_device_memory()
        for rec, bytes_step, flops in ((ours, (body + vocab * C) * 2 + kv, 2.0 * B * P * body + B * att_flops),
                                       (like, like_bytes, 2.0 * B * P * like_body + B * like_att)):
            rec.update(prefill_tokens_per_s=B * P / rec["prefill_ms"] * 1e3, decode_tokens_per_s=B / rec["ms_per_decode_step"] * 1e3,
                       e2e_tokens_per_s=B * (P + N) / rec["e2e_ms"] * 1e3,
                       prefill_frac=flops / rec["prefill_ms"] / 1e9 / peaks["bf16_tflops"],
                       decode_frac=bytes_step / rec["ms_per_decode_step"] / 1e6 / peaks["hbm_gbs"])
        records.append({"size": name, "width": C, "ff": F, "heads": H, "kv_heads": G, "params_body": body, args.mode: ours,
                        like_name: {**like, "ffn": ffn}})
    mid = records[len(records) // 2][args.mode]
    ms = mid["prefill_ms"] + mid["ms_per_decode_step"] * (N - 1)
    print(json.dumps({
        "impl": "ours", "metric": SERVING_METRIC.format(design), "value": B * (P + N) / ms * 1e3, "unit": "tokens/s", "n_gpus": 1,
        "steps": K, "warmup": W, "ms_per_step": ms, "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic (uniform random prompt ids, random weights)",
        "config": {"model": f"{design}, 4 layers", "global_batch": B, "seq_len": P + N, "parallelism": "1 GPU",
                   "l2": "weights and activations of a step exceed the 126 MB L2; no flush needed"},
        "clocks": mid["clocks"], "gpu_launches": launches_total,
        "e2e": {"value": mid["e2e_tokens_per_s"], "unit": "tokens/s", "h2d_bytes_per_step": B * P * 4 + 2 * B * 4,
                "d2h_bytes_per_step": B * N * 4}, "sizes": records}))
    return 0


def _free_device_memory():
    import gc

    import torch

    gc.collect()
    torch.cuda.synchronize()
    torch.cuda.empty_cache()


def _torch_train_arm(args, cfg, tp, K, W, rank, local_rank, dist_barrier, dist):
    """The PyTorch (+cuBLAS, flash SDPA, NCCL) implementation of the same step on the same GPUs: the number to beat on
    this machine. Returns `(adapter with step / step_device / synthetic_tokens / tokens_per_step, trainer)`."""
    import torch

    sys.path.insert(0, os.path.join(os.path.dirname(os.path.abspath(__file__)), "baseline"))
    if args.mode == "pipeline":
        from torch_pipeline import TorchPipelineTrainer

        tt = TorchPipelineTrainer(cfg, stages=min(args.stages, args.gpus), micro_batches=args.micro_batches)
        tt.graph_note = "eager (1F1B schedule issued from Python)"
    else:
        from torch_decoder import TorchTrainer

        tt = TorchTrainer(cfg, micro_batches=args.micro_batches, recompute=args.recompute,
                          cuda_graph=not args.no_cuda_graphs)

    class _Adapter:
        tokens_per_step = tt.tokens_per_step
        prune_recompute = False

        class session:
            h2d_bytes = 0
            d2h_bytes = 0

        def synthetic_tokens(self, seed=0):
            # every process of one replica (its TP ranks, or its pipeline stages) sees the same tokens
            per_replica = min(args.stages, args.gpus) if args.mode == "pipeline" else max(tp, 1)
            g = torch.Generator().manual_seed(seed + rank // per_replica)
            return torch.randint(0, cfg.vocab_size, (args.micro_batches, 1, 1, cfg.seq_len + 1), generator=g,
                                 dtype=torch.int32).pin_memory()

        def step(self, t):
            _Adapter.session.h2d_bytes += t.numel() * 4
            _Adapter.session.d2h_bytes += 4
            return tt.step(t)

        def step_device(self, t):
            return tt.step_device(t)

    return _Adapter(), tt


def _time_steps(trainer, K, W, barrier, local_rank, dist, native=None, e2e=True, pipeline_stages=0):
    """W untimed steps, then K steps timed on the device (inputs resident, CUDA events, max over ranks) and, if `e2e`, K
    more through the public `step` call (tokens from pinned host memory in, losses out), by wall clock between
    barriers."""
    import torch

    host_tokens = [trainer.synthetic_tokens(seed=i) for i in range(W + K)]
    dev_tokens = [t.cuda(non_blocking=True) for t in host_tokens]
    losses = []
    for i in range(W):
        losses.append(trainer.step(host_tokens[i]))
    losses = [l if l is not None else float("nan") for l in losses]
    launches0 = native.LAUNCHES["count"] if native is not None else 0
    start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    with ClockSampler(local_rank) as clocks:
        barrier()
        start.record()
        for i in range(K):
            trainer.step_device(dev_tokens[W + i])
        end.record()
        barrier()
    dev_ms = start.elapsed_time(end)
    launches = (native.LAUNCHES["count"] - launches0) if native is not None else 0
    if native is not None:
        native.check_gemm_errors()
    e2e_s, h2d, d2h = float("nan"), 0, 0
    if e2e:
        h2d0, d2h0 = trainer.session.h2d_bytes, trainer.session.d2h_bytes
        barrier()
        t1 = time.perf_counter()
        for i in range(K):
            losses.append(trainer.step(host_tokens[W + i]))
        barrier()
        e2e_s = time.perf_counter() - t1
        h2d = (trainer.session.h2d_bytes - h2d0) // K
        d2h = (trainer.session.d2h_bytes - d2h0) // K
    if pipeline_stages and dist is not None:
        box = [losses]
        dist.broadcast_object_list(box, src=pipeline_stages - 1)  # the last slot of replica 0 computes the loss
        losses = box[0]
    times = torch.tensor([dev_ms, e2e_s * 1e3], dtype=torch.float64, device="cuda")
    if dist is not None:
        dist.all_reduce(times, op=dist.ReduceOp.MAX)
    return {"dev_ms": float(times[0]), "e2e_ms": float(times[1]), "launches": int(launches), "h2d": int(h2d),
            "d2h": int(d2h), "losses": losses, "clocks": clocks.summary()}


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=4)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference", "torch"])
    ap.add_argument("--model", default="gptj_6b")
    ap.add_argument("--micro-batches", type=int, default=16)
    ap.add_argument("--micro-batch-size", type=int, default=1)
    ap.add_argument("--layers", type=int, default=0, help="override the layer count (diagnostics only; such a run is "
                                                         "labelled and is not the headline configuration)")
    ap.add_argument("--mode", default="train", choices=["train", "decode", "pipeline", "dunelix", "zirunex"],
                    help="train: the training step (default, headline), followed by the PyTorch arm of the same step and "
                         "the int4 decode benchmark as secondary records; decode: int4 greedy generation, TP over all "
                         "GPUs; pipeline: pipeline x data parallel training (--stages device slots per replica); "
                         "dunelix, zirunex: prefill and decoding of that design's layers at several sizes, beside the int4 "
                         "GPT-J generator / beside Dunelix (one GPU; --model w2048|w4096|w8192 runs one size)")
    ap.add_argument("--tp", type=int, default=0, help="train mode: tensor-parallel width (default min(gpus, 4))")
    ap.add_argument("--stages", type=int, default=4, help="pipeline mode: device slots (GPUs) per replica")
    ap.add_argument("--sequence-parallel", action="store_true",
                    help="train mode: shard the residual stream over the tokens inside the TP group")
    ap.add_argument("--recompute", action="store_true",
                    help="train / pipeline mode, both arms: run each block's forward pass a second time in the backward "
                         "pass instead of keeping its activations (the reference needs this on IPUs; 180 GB of HBM do "
                         "not: a micro-batch of 2048 tokens keeps about 6 GB at TP1, the default keeps them)")
    ap.add_argument("--no-recompute", action="store_true", help="the default since activations fit; kept for old commands")
    ap.add_argument("--prune-recompute", action="store_true",
                    help="with --recompute: the recomputed forward pass of a block leaves out the ops that only lead "
                         "to the block's output (also XL_PRUNE_RECOMPUTE=1); the gradients are bit-identical")
    ap.add_argument("--batch", type=int, default=16, help="decode mode: sequences per batch")
    ap.add_argument("--prompt-len", type=int, default=512)
    ap.add_argument("--new-tokens", type=int, default=128)
    ap.add_argument("--no-cuda-graphs", action="store_true")
    ap.add_argument("--no-baseline", action="store_true",
                    help="train mode, --impl ours: skip the PyTorch arm that is otherwise timed first on the same GPUs")
    ap.add_argument("--no-decode", action="store_true",
                    help="train mode, --impl ours: skip the int4 decode benchmark that otherwise follows as a secondary record")
    ap.add_argument("--profile-ops", action="store_true",
                    help="diagnostics, --impl ours: after the timed regions run one more step with per-op CUDA-event timing "
                         "(eagerly, no graph replay) and print the per-op totals as a second line starting with PROFILE")
    ap.add_argument("--emulate-tp", type=int, default=0,
                    help="diagnostics: run ONE rank's shard shapes of a K-way tensor-parallel layout (heads, ffn and "
                         "vocabulary divided by K, no collectives) to separate kernel time from communication")
    ap.add_argument("--torch-dense", action="store_true",
                    help="decode mode, --impl torch: keep a bf16 copy of every weight instead of de-quantising per call")
    args = ap.parse_args()
    if args.impl == "reference":
        return run_reference(args)
    if args.mode == "decode":
        return run_decode(args)
    if args.mode in ("dunelix", "zirunex"):
        return run_serving(args)

    import torch

    from popxl_addons_b200.models.decoder import DecoderConfig

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if world != args.gpus:
        if world == 1 and args.gpus > 1:
            raise SystemExit("launch with torch.distributed.run --nproc-per-node N for --gpus N > 1")
    torch.cuda.set_device(local_rank)
    tp, dp = layout_for(args.gpus)
    if args.tp:
        tp, dp = args.tp, args.gpus // args.tp
    pipeline = args.mode == "pipeline"
    stages = 0
    if pipeline:
        stages = min(args.stages, args.gpus)
        tp, dp = 1, args.gpus // stages
        if args.model == "gptj_6b":
            args.model = "llama2_7b"
        if args.micro_batches == 16:
            args.micro_batches = 32
    cfg = getattr(DecoderConfig, args.model)(tp=tp, dp=dp)
    if args.layers:
        cfg.layers = args.layers
    if args.emulate_tp:
        _shrink(cfg, args.emulate_tp)
    cfg.sequence_parallel = bool(args.sequence_parallel)
    W = max(args.warmup, 3)
    K = args.steps
    headline = (not args.layers and not args.emulate_tp and args.model == "gptj_6b" and not pipeline and not args.tp
                and args.micro_batch_size == 1 and args.micro_batches == 16)
    dist_holder = {"dist": None}

    def barrier():
        d = dist_holder["dist"]
        if d is not None:
            d.barrier()
        torch.cuda.synchronize()

    def current_dist():
        d = torch.distributed if (world > 1 and torch.distributed.is_initialized()) else None
        dist_holder["dist"] = d
        return d

    # ---- the PyTorch arm of the same step, timed first on the same GPUs (its memory is released afterwards) ----------
    baseline = None
    run_baseline = args.impl == "ours" and not args.no_baseline and not args.emulate_tp \
        and not args.sequence_parallel
    if args.impl == "torch" or run_baseline:
        t0 = time.perf_counter()
        adapter, tt = _torch_train_arm(args, cfg, tp, K, W, rank, local_rank, barrier, None)
        torch_setup_s = time.perf_counter() - t0
        dist = current_dist()
        kb = K if args.impl == "torch" else min(K, 3)
        res = _time_steps(adapter, kb, W, barrier, local_rank, dist, e2e=True,
                          pipeline_stages=stages if pipeline else 0)
        res.update(steps=kb, setup_s=torch_setup_s, tokens=adapter.tokens_per_step, graph_note=tt.graph_note)
        baseline = res
        if args.impl == "ours":
            del adapter, tt
            _free_device_memory()

    native = None
    ours = None
    setup_s = 0.0
    trainer = None
    if args.impl == "ours":
        t0 = time.perf_counter()
        from popxl_addons_b200.ops import native

        native.STRICT[0] = True  # a hot op that falls back to the library implementation on this GPU is an error
        if pipeline:
            from popxl_addons_b200.models.pipeline_trainer import PipelineTrainer

            trainer = PipelineTrainer(cfg, stages=stages, micro_batches=args.micro_batches,
                                      micro_batch_size=args.micro_batch_size, device="cuda", seed=0, lr=1e-4,
                                      recompute=args.recompute,
                                      prune_recompute=True if args.prune_recompute else None)
        else:
            from popxl_addons_b200.models.trainer import DecoderTrainer

            trainer = DecoderTrainer(cfg, micro_batches=args.micro_batches, micro_batch_size=args.micro_batch_size,
                                     device="cuda", seed=0, lr=1e-4, recompute=args.recompute,
                                     prune_recompute=True if args.prune_recompute else None,
                                     cuda_graphs=not args.no_cuda_graphs)
        setup_s = time.perf_counter() - t0
        dist = current_dist()
        ours = _time_steps(trainer, K, W, barrier, local_rank, dist, native=native, e2e=True,
                           pipeline_stages=stages if pipeline else 0)
        ours["kernels"] = dict(native.LAUNCHES["by_kernel"])
        ours["fallbacks"] = dict(native.FALLBACKS)
        ours["tokens"] = trainer.tokens_per_step
        ours["prune"] = bool(getattr(trainer, "prune_recompute", False))
        ours["peak_gb"] = round(torch.cuda.max_memory_allocated() / 2 ** 30, 1)
        if args.profile_ops:
            trainer.session.start_profile()
            trainer.step(trainer.synthetic_tokens(seed=99))
            prof = trainer.session.profile_summary()
            if rank == 0:
                total = sum(v["ms"] for v in prof.values())
                print("PROFILE " + json.dumps({"total_ms": total, "ops": {k: {"count": v["count"], "ms": round(v["ms"], 2)}
                                                                          for k, v in list(prof.items())[:40]}}))
    main_res = ours if args.impl == "ours" else baseline
    dist = current_dist()

    # ---- secondary record: int4 greedy generation, tensor parallel over all GPUs (the second headline metric) ----------
    decode = None
    if args.impl == "ours" and headline and not args.no_decode:
        del trainer
        _free_device_memory()
        dargs = argparse.Namespace(**vars(args))
        dargs.mode, dargs.steps, dargs.warmup = "decode", min(K, 2), 3
        before = dict(native.LAUNCHES["by_kernel"])
        dec_lines = {}
        for impl, dense in (("torch", True), ("ours", False)):
            dargs.impl, dargs.torch_dense = impl, dense
            try:
                dec_lines[impl] = run_decode(dargs, standalone=False)
            except Exception as e:  # the secondary record must not take the headline down with it
                dec_lines[impl] = {"error": f"{type(e).__name__}: {e}"} if rank == 0 else None
        if rank == 0:
            d_ours, d_torch = dec_lines["ours"], dec_lines["torch"]
            if d_ours and "kernels" in d_ours:
                d_ours["kernels"] = {k: v - before.get(k, 0) for k, v in d_ours["kernels"].items()
                                     if v - before.get(k, 0) > 0}
            decode = d_ours
            if d_ours and d_torch and "value" in d_ours and "value" in d_torch:
                decode["vs_baseline"] = d_ours["value"] / d_torch["value"]
                decode["baseline"] = {"impl": "PyTorch + cuBLAS, CUDA-graph-replayed decode step, bf16 copy of every "
                                              "weight (4x the memory of the int4 model: the upper bound of the library path)",
                                      "value": d_torch["value"], "ms_per_step": d_torch["ms_per_step"],
                                      "ms_per_decode_step": d_torch["ms_per_decode_step"], "steps": d_torch["steps"]}
            elif d_torch:
                decode = decode or {}
                decode["baseline"] = d_torch

    if rank == 0:
        tokens = main_res["tokens"]
        kk = main_res.get("steps", K)
        value = tokens * kk / (main_res["dev_ms"] / 1e3)
        e2e_value = tokens * kk / (main_res["e2e_ms"] / 1e3)
        # model FLOPs only: 6 x parameters x tokens plus the attention products; a recomputed forward pass is not counted
        flops_per_token = 6 * cfg.param_count() + 6 * cfg.layers * cfg.seq_len * cfg.heads * cfg.head_dim
        vs, vs_detail = None, None
        if args.impl == "ours" and baseline is not None:
            bval = baseline["tokens"] * baseline["steps"] / (baseline["dev_ms"] / 1e3)
            be2e = baseline["tokens"] * baseline["steps"] / (baseline["e2e_ms"] / 1e3)
            vs = value / bval
            vs_detail = {"impl": "PyTorch + cuBLAS + flash SDPA + NCCL, same step on the same GPUs in this run "
                                 + ("(baseline/torch_pipeline.py, 1F1B)" if pipeline else "(baseline/torch_decoder.py)"), "value": bval, "ratio": vs, "e2e_value": be2e,
                         "e2e_ratio": e2e_value / be2e, "steps": baseline["steps"], "warmup": W,
                         "ms_per_step": baseline["dev_ms"] / baseline["steps"], "cuda_graph": baseline["graph_note"],
                         "clocks": baseline["clocks"]}
        line = {
            "impl": args.impl, "metric": PIPELINE_METRIC if pipeline else METRIC, "value": value, "unit": "tokens/s",
            "n_gpus": args.gpus, "steps": kk, "warmup": W, "ms_per_step": main_res["dev_ms"] / kk,
            "higher_is_better": True,
            # tensor parallel up to 4 GPUs keeps the global batch (strong scaling); beyond that data-parallel replicas
            # are added and the global batch grows with them (weak scaling)
            "scaling": "strong" if dp == 1 else "weak",
            "scaling_note": f"global batch = {args.micro_batches * args.micro_batch_size} sequences x dp ({dp}); "
                            f"tp{tp} splits one replica's work",
            "vs_baseline": vs, "vs_baseline_detail": vs_detail,
            "dtype": "bf16", "data": "synthetic (uniform random token ids, random-init weights)",
            "config": {"model": f"{args.model} ({cfg.layers} layers, hidden {cfg.hidden}, {cfg.heads} heads x "
                                f"{cfg.head_dim}, ffn {cfg.ffn}, vocab {cfg.vocab_size})",
                       "global_batch": args.micro_batches * args.micro_batch_size * dp, "seq_len": cfg.seq_len,
                       "parallelism": (f"pp{stages}xdp{dp}" if pipeline else f"tp{tp}xdp{dp}"),
                       "micro_batches": args.micro_batches, "micro_batch_size": args.micro_batch_size,
                       "optimizer": "AdamW, fp32 master weights + fp32 moments" +
                                    (", state sharded over dp (RTS)" if dp > 1 else ""),
                       "recompute": ("per layer" + (", second forward pass reduced to what the backward pass reads"
                                                    if main_res.get("prune") else "")) if args.recompute
                       else "none (activations kept: they fit in HBM; both arms)",
                       "l2": "each step streams >100 GB of weights, optimizer state and activations, far beyond the "
                             "126 MB L2; no flush needed",
                       "emulate_tp": args.emulate_tp or None, "sequence_parallel": bool(args.sequence_parallel),
                       "headline": headline},
            "clocks": main_res["clocks"],
            "peak_memory_gb": main_res.get("peak_gb", round(torch.cuda.max_memory_allocated() / 2 ** 30, 1)),
            "e2e": {"value": e2e_value, "unit": "tokens/s", "ms_per_step": main_res["e2e_ms"] / kk,
                    "h2d_bytes_per_step": main_res["h2d"], "d2h_bytes_per_step": main_res["d2h"]},
            "gpu_launches": main_res["launches"],
            "kernels": main_res.get("kernels", {}),
            "fallbacks": main_res.get("fallbacks", {}),
            "model_tflops_per_gpu": flops_per_token * value / args.gpus / 1e12,
            "flops_note": "model FLOPs (6 x parameters + attention) per token; recomputed passes are not counted",
            "loss_first_last": [main_res["losses"][0], main_res["losses"][-1]],
            "setup_seconds": setup_s if args.impl == "ours" else baseline["setup_s"], "mode": args.mode,
            "secondary": decode,
        }
        if args.impl == "torch":
            line["config"]["cuda_graph"] = baseline["graph_note"]
        print(json.dumps(line))
    _shutdown(dist)
    return 0


if __name__ == "__main__":
    sys.exit(main())
