#!/usr/bin/env python3
"""Decode and prefill throughput at Qwen3-8B layer sizes with random weights, on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--layers L] [--shape 8b|0.6b|32b] [--impl ours|reference]
    python bench.py --workload mixed [--shape 0.6b|8b]     # 64 requests, continuous batching
    python bench.py --kernels                               # single kernels at serving sizes
    python bench.py --kernels --attn 16,8,64                # the attention kernels at another head layout
    python bench.py --ablate                                # a decode step with one kind of kernel left out at a time
    python bench.py --compare tidarax [--size 1k|4k]        # the Tidarax design beside Qwen3 at equal layer sizes
    python bench.py --compare dufitar [--size 1k|4k]        # the Dufitar design beside Qwen3 at equal layer sizes
    python bench.py --compare gulipel [--size 1k|4k]        # the Gulipel design beside Tidarax at equal layer sizes
    python bench.py --compare mikutar [--size 1k|4k]        # the Mikutar design beside Dufitar at equal layer sizes
    python bench.py --compare napuzen [--size 1k|4k]        # the Napuzen design beside Dufitar and Gulipel at equal layer sizes
    python bench.py --compare dalalix [--size 1k|4k]        # the Dalalix design beside Mikutar and Gulipel at equal layer sizes

Prints ONE JSON line.  ``value`` is decoded tokens per second at batch 8 and the context length
of the configuration (a "step" is one decode step of the whole batch), timed on the device with
CUDA events around exactly K steps; ``e2e`` is the same through the Python entry point
(``Engine.step``: host token ids in through pinned memory every step, sampled ids read back every
step).  ``prefill`` times one step of 2,048 prompt tokens; ``roofline`` divides the bytes a decode
step must read (every weight once, the cache of the live requests) by its time; ``points`` holds
decode at batch 1 and 64 at the same context, and ``baseline_b1/8/64``: decode tokens per second
over 256 steps after a 2,048-token prompt (context 2,048 -> 2,304).  Fractions are given against the
measured peaks (MEASURED_PEAKS.json beside this file, when present) and, as ``frac_nominal``, against
the nominal 8 TB/s and 2.25 PFLOP/s.  The logits of the first prefill and of the last decode step
are checked to be finite (their largest magnitudes stand in ``config``).

``--workload mixed``: 64 requests with prompt lengths uniform in 16..2,048 (seeded), 256 new tokens
each, through ``Engine.generate_sync``: decoded and total tokens per second, steps, the distribution
of step times and the number of preemptions, as one JSON line (the reference's batch test,
src/main.rs:103-115, 502-555, is the counterpart).
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

# Layer sizes of the headline configuration (Qwen3-8B shape).
CONFIG = dict(
    architectures=["Qwen3ForCausalLM"], vocab_size=151936, hidden_size=4096, intermediate_size=12288,
    num_hidden_layers=36, num_attention_heads=32, num_key_value_heads=8, head_dim=128,
    rms_norm_eps=1e-6, rope_theta=1000000.0, max_position_embeddings=40960,
    tie_word_embeddings=False, sliding_window=None,
)
# The other two published shapes, for --shape: what differs from the headline configuration.
SHAPES = {
    "8b": {},
    "0.6b": dict(hidden_size=1024, intermediate_size=3072, num_hidden_layers=28, num_attention_heads=16,
                 tie_word_embeddings=True),
    "32b": dict(hidden_size=5120, intermediate_size=25600, num_hidden_layers=64, num_attention_heads=64),
}
CONTEXT = 4096
PREFILL_TOKENS = 2048
NOMINAL_HBM_GBS = 8000.0
NOMINAL_BF16_TFLOPS = 2250.0
PAGE = 16
SETTLE = 24   # untimed decode steps between a prefill burst and any timed decode step, beside --warmup


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        with open(path) as f:
            p = json.load(f)
        return dict(hbm_gbs=float(p["hbm_gbs"]), bf16_tflops=float(p["bf16_tflops"]), source="measured")
    return dict(hbm_gbs=6650.0, bf16_tflops=1590.0, source="fallback")


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region is timed."""

    FIELDS = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples = []
        self.proc = None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits", "-lms", "10"],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.samples.append((time.time(), line.strip()))

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self, t0: float, t1: float):
        mhz, mx, reasons = [], 0, set()
        names = ("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap")
        for t, line in self.samples:
            if t < t0 or t > t1 + 0.2:
                continue
            parts = [p.strip() for p in line.split(",")]
            try:
                mhz.append(float(parts[0]))
                mx = max(mx, float(parts[1]))
            except (ValueError, IndexError):
                continue
            for name, val in zip(names, parts[2:6]):
                if val.lower().startswith("active"):
                    reasons.add(name)
        mhz.sort()
        return {"sm_mhz": mhz[len(mhz) // 2] if mhz else None, "sm_max_mhz": mx or None,
                "reasons": sorted(reasons), "samples": len(mhz)}


def reference_arm():
    print(json.dumps({"impl": "reference", "unavailable":
                      "the reference is a Rust crate (no setup.py/pyproject.toml; pip: 'not installable'); "
                      "no Rust toolchain and no network on this machine"}))
    return 0


def check_finite(logits, what: str) -> float:
    """A benchmark line must not come from a model that computes nonsense: every logit finite, and
    not all of them alike.  Returns the largest magnitude."""
    import torch
    v = logits.float()
    if not bool(torch.isfinite(v).all()):
        raise SystemExit(f"bench.py: the logits of {what} are not finite")
    if float(v.max() - v.min()) == 0.0:
        raise SystemExit(f"bench.py: the logits of {what} are all equal")
    return round(float(v.abs().max()), 3)


def mixed_workload(args, cfg, full, pk) -> int:
    """Continuous batching: ``--requests`` requests, prompt lengths uniform in [16, 2048] (seeded), 256 new
    tokens each, greedy, through the Python entry point.  One untimed pass (graphs are captured, buffers
    sized), then the timed one with fresh prompts of the same lengths."""
    import numpy as np
    import torch
    from xinfer_b200.config import EngineConfig
    from xinfer_b200.engine.llm import Engine
    from xinfer_b200.engine.runner import ModelRunner
    from xinfer_b200.sampling import SamplingParams

    N, new_tokens = args.requests, 256
    max_len = 2048 + new_tokens + 64
    runner = ModelRunner.random(cfg, seed=0, dtype="bfloat16", block_size=PAGE, num_blocks=N * (max_len // PAGE + 1),
                                max_num_seqs=N, max_model_len=max_len)
    engine = Engine(EngineConfig(weight_path="(random)", block_size=PAGE, max_num_seqs=N, max_num_batched_tokens=8192,
                                 prefill_chunk_size=2048, max_model_len=max_len, disable_cuda_graph=args.no_graph),
                    "bf16", runner=runner)
    rng = np.random.default_rng(0)
    V = cfg["vocab_size"]
    lens = rng.integers(16, 2049, size=N)
    sp = SamplingParams(temperature=0.0, max_tokens=new_tokens, ignore_eos=True)
    clocks = ClockSampler()
    clocks.start()
    result = None
    for timed in (False, True):
        prompts = [rng.integers(0, V, size=int(n)).tolist() for n in lens]
        before = dict(engine.stats)
        torch.cuda.synchronize()
        t0 = time.time()
        ids = [engine.add_request(p, sp) for p in prompts]
        step_ms = []
        last = t0
        while any(i in engine._live for i in ids):
            engine.step()
            now = time.time()
            step_ms.append((now - last) * 1e3)
            last = now
        torch.cuda.synchronize()
        t1 = time.time()
        outs = [engine._done.pop(i) for i in ids]
        if any(o.error for o in outs) or any(o.decoded_length != new_tokens for o in outs):
            raise SystemExit("bench.py: the mixed workload did not finish every request")
        if timed:
            st = {k: engine.stats[k] - before[k] for k in before}
            decoded, prompt = sum(o.decoded_length for o in outs), int(lens.sum())
            step_ms.sort()
            pick = lambda q: round(step_ms[min(len(step_ms) - 1, int(q * len(step_ms)))], 3)
            result = {
                "metric": f"decoded tok/s, continuous batching of {N} requests (Qwen3-{args.shape.upper()} shape)",
                "value": round(decoded / (t1 - t0), 1), "unit": "tokens/s", "total_tok_s": round((decoded + prompt) / (t1 - t0), 1),
                "n_gpus": 1, "seconds": round(t1 - t0, 3), "steps": st["steps"], "steps_decided_ahead": st["steps_decided_ahead"],
                "preemptions": st["preemptions"], "step_ms": {"p50": pick(0.5), "p90": pick(0.9), "p99": pick(0.99), "max": round(step_ms[-1], 3)},
                "prompt_tokens": prompt, "decoded_tokens": decoded, "dtype": "bf16", "impl": "ours",
                "data": "synthetic (random weights, seeded uniform token ids)", "higher_is_better": True,
                "config": {"model": f"Qwen3-{args.shape.upper()} shape", "layers": cfg["num_hidden_layers"],
                           "layers_of_config": full["num_hidden_layers"], "requests": N, "prompt_len": "uniform 16..2048",
                           "new_tokens": new_tokens, "page_size": PAGE, "max_num_batched_tokens": 8192,
                           "prefill_chunk_size": 2048, "cuda_graph": not args.no_graph},
                "clocks": clocks.summary(t0, t1),
            }
    clocks.stop()
    print(json.dumps(result))
    return 0


# Layer sizes for --compare: a Tidarax model and a Qwen3 model of the same width, heads, head size and
# feed-forward size (the recurrence as wide as the model, experts a quarter of the dense feed-forward each).
COMPARE_SIZES = {
    "1k": dict(hidden=1024, heads=16, kv_heads=8, head_dim=128, intermediate=3072, experts=8, expert_ff=768, top=2),
    "4k": dict(hidden=4096, heads=32, kv_heads=8, head_dim=128, intermediate=12288, experts=8, expert_ff=3072, top=2),
}


def tidarax_config(z: dict, layers: int, vocab: int) -> dict:
    left = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=z["head_dim"], vdim=z["head_dim"], scale=z["head_dim"] ** -0.5,
                rot=dict(dims=z["head_dim"], base=500000.0, scaling=dict(factor=8.0, low=1.0, high=4.0, original=8192)))
    mixer = dict(left=left, left_scale=1.0, right=dict(width=z["hidden"]), right_scale=1.0)
    dense = dict(kind="dense", ff=z["intermediate"])
    moe = dict(kind="moe", expert=dict(ff=z["expert_ff"]), router=dict(experts=z["experts"], top=z["top"]))
    return dict(architecture="Tidarax", vocab=vocab, width=z["hidden"], norm=dict(eps=1e-6),
                layers=[dict(type="parallel", mixer=mixer, mlp=dense if i % 2 == 0 else moe) for i in range(layers)])


# The latent layers of --compare dufitar: what a token leaves in the cache, and the rotated part of a head.
LATENT_SIZES = {"1k": dict(kv_rank=256, rot_dim=32), "4k": dict(kv_rank=512, rot_dim=64)}
# windows of --compare dufitar: wider than the benchmark's context, so that its attention does the work of
# the Qwen3 model's (which sees every earlier key)
COMPARE_WINDOW = 4096


def dufitar_config(z: dict, lat: dict, layers: int, vocab: int) -> dict:
    d = z["head_dim"]
    attn = dict(type="attention", mlp=dict(kind="dense", ff=z["intermediate"]),
                mixer=dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=d, vdim=d, scale=d ** -0.5, mask=dict(size=COMPARE_WINDOW),
                           rot=dict(dims=d // 2, base=1000000.0, scaling=dict(factor=8.0, original=8192, fast=16.0, slow=2.0))))

    def latent(kv_from=None):
        m = dict(heads=z["heads"], dim=d, rot_dim=lat["rot_dim"], vdim=d, kv_rank=lat["kv_rank"],
                 scale=(d + lat["rot_dim"]) ** -0.5, mask=dict(size=COMPARE_WINDOW), rot=dict(dims=lat["rot_dim"], base=100000.0))
        if kv_from is not None:
            m["kv_from"] = kv_from
        return dict(type="latent_attention", mixer=m, mlp=dict(kind="dense", ff=z["intermediate"]))

    out = []
    for i in range(layers):      # attention, latent, attention, latent reading the rows of the latent layer before it
        out.append(attn if i % 2 == 0 else latent(i - 2 if i % 4 == 3 else None))
    return dict(architecture="Dufitar", vocab=vocab, width=z["hidden"], norm=dict(eps=1e-6), residual_mult=0.5,
                embedding=dict(scale=2.0), layers=out)


# The recurrent layers of --compare gulipel: a state-space mixer twice as wide as the model in heads of 64 channels
# with a state of 128 per channel, and a gated delta rule with as many heads as the attention beside it.
def gulipel_sizes(z: dict) -> dict:
    ss_heads = 2 * z["hidden"] // 64
    return dict(ss_heads=ss_heads, ss_head_dim=64, ss_state=128, ss_groups=max(1, ss_heads // 16), conv=4,
                delta_heads=z["heads"], delta_kv_heads=z["heads"], delta_dim=z["head_dim"], delta_vdim=z["head_dim"], rank=64)


def gulipel_config(z: dict, layers: int, vocab: int, max_positions: int) -> dict:
    g, d = gulipel_sizes(z), z["head_dim"]
    dense = dict(kind="dense", ff=z["intermediate"])
    ssm = dict(heads=g["ss_heads"], vdim=g["ss_head_dim"], state=g["ss_state"], groups=g["ss_groups"], conv=g["conv"],
               norm_groups=g["ss_groups"])
    par = dict(left=dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=d, vdim=d, scale=d ** -0.5, q_temp=dict(coef=0.25, every=512)),
               right=dict(heads=g["delta_heads"], kv_heads=g["delta_kv_heads"], dim=g["delta_dim"], vdim=g["delta_vdim"], conv=g["conv"],
                          decay_rank=g["rank"], gate_rank=g["rank"]))
    # state-space layers with a parallel layer every other one: as many attention layers per model as a Tidarax
    # model of half the depth, the rest recurrent
    out = [dict(type="parallel", mixer=par, mlp=dense) if i % 2 == 1 else dict(type="mamba2" if i % 4 == 0 else "mamba2_2", mixer=ssm, mlp=dense)
           for i in range(layers)]
    return dict(architecture="Gulipel", vocab=vocab, width=z["hidden"], norm=dict(eps=1e-6), max_positions=max_positions,
                logit_softcap=40.0, embedding=dict(scale=z["hidden"] ** 0.5, bigram=dict(buckets=100003, mul_prev=8191, mul_cur=31)),
                token_side=dict(dim=64), layers=out)


# --compare mikutar: windowed attention / dense, windowed / experts, windowed / dense, chunked with capped scores /
# experts; windows and chunks wider than the benchmark's context; experts of a quarter of the dense width in four
# groups of which two are kept, beside an expert of the same size that every token runs.  ``loop``: the first three
# layers run twice (seven layer runs) where it is set.
def mikutar_config(z: dict, layers: int, vocab: int, loop: bool = False) -> dict:
    d = z["head_dim"]
    common = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=d, vdim=d, scale=d ** -0.5, mask=dict(size=COMPARE_WINDOW))
    attn = dict(type="attention", mixer=dict(common, rot=dict(dims=d // 2, base=500000.0)))
    attn2 = dict(type="attention_2", mixer=dict(common, softcap=40.0))
    dense = dict(kind="dense", ff=z["intermediate"])
    moe = dict(kind="moe", expert=dict(ff=z["expert_ff"], limit=7.0), shared=dict(ff=z["expert_ff"], limit=7.0),
               router=dict(experts=z["experts"], top=z["top"], groups=dict(count=4, keep=2)))
    out = [dict(attn2 if i % 4 == 3 else attn, mlp=moe if i % 2 else dense) for i in range(layers)]
    cfg = dict(architecture="Mikutar", vocab=vocab, width=z["hidden"], norm=dict(eps=1e-6), logit_softcap=30.0, layers=out)
    if loop and layers > 1:
        cfg["loop"] = dict(start=0, stop=layers - 1, times=2)
    return cfg


# --compare napuzen: linear attention / dense, latent attention without positions / experts, linear attention / dense,
# latent attention with a rotated part / experts; the linear attention with as many heads as the other designs' attention,
# latents and experts of the sizes above, windows wider than the benchmark's context, queries through a latent of three
# times the cached one's size.
def napuzen_config(z: dict, lat: dict, layers: int, vocab: int) -> dict:
    H, d, r = z["heads"], z["head_dim"], lat["kv_rank"]
    gla = dict(type="gla", mixer=dict(heads=H, dim=d, vdim=d, tau=8.0))
    rot = dict(dims=lat["rot_dim"], base=100000.0, scaling=dict(factor=4.0, original=8192, fast=16.0, slow=2.0))
    latent = dict(type="latent_attention", mixer=dict(heads=H, dim=d, rot_dim=lat["rot_dim"], vdim=d, q_rank=3 * r, kv_rank=r,
                                                      scale=(d + lat["rot_dim"]) ** -0.5, rot=rot))

    def latent2(kv_from=None):
        m = dict(heads=H, dim=d, vdim=d, kv_rank=r, scale=d ** -0.5, mask=dict(size=COMPARE_WINDOW))
        if kv_from is not None:
            m["kv_from"] = kv_from
        return dict(type="latent_attention_2", mixer=m)
    dense = dict(kind="dense", ff=z["intermediate"], limit=7.0)
    moe = dict(kind="moe", expert=dict(ff=z["expert_ff"]), shared=dict(ff=z["expert_ff"]),
               router=dict(experts=z["experts"], top=z["top"], scale=1.5))
    out = []
    for i in range(layers):
        mixer = gla if i % 2 == 0 else (latent if i % 4 == 3 else latent2(i - 4 if i % 8 == 5 else None))
        out.append(dict(mixer, mlp=moe if i % 2 else dense))
    return dict(architecture="Napuzen", vocab=vocab, width=z["hidden"], norm=dict(eps=1e-6), canon=dict(taps=4), logit_scale=0.8,
                layers=out)


# --compare dalalix: convolved attention, attention with biases, attention beside a matrix memory, convolved attention;
# experts in every layer, four groups of which two are kept; four residual streams; a window wider than the benchmark's
# context that keeps the first 64 tokens; the memory with as many heads as the attention.
def dalalix_config(z: dict, layers: int, vocab: int) -> dict:
    d = z["head_dim"]
    common = dict(heads=z["heads"], kv_heads=z["kv_heads"], dim=d, vdim=d, scale=d ** -0.5)
    mlp = dict(kind="moe", expert=dict(ff=z["expert_ff"], limit=7.0),
               router=dict(experts=z["experts"], top=z["top"], groups=dict(count=4, keep=2)))
    conv = dict(type="attention", mixer=dict(common, conv=4), mlp=mlp)
    biased = dict(type="attention_2", mixer=common, mlp=mlp)
    left = dict(common, mask=dict(size=COMPARE_WINDOW, keep_first=64), rot=dict(dims=d // 2, base=500000.0))
    par = dict(type="parallel", mlp=mlp, mixer=dict(left=left, left_scale=0.75, right_scale=0.5,
                                                    right=dict(heads=z["heads"], dim=d, vdim=d, gate_cap=15.0)))
    return dict(architecture="Dalalix", vocab=vocab, width=z["hidden"], norm=dict(eps=1e-6), streams=4, logit_softcap=30.0,
                embedding=dict(bigram=dict(buckets=50021, mul_prev=8191, mul_cur=127)),
                layers=[(conv, biased, par, conv)[i % 4] for i in range(layers)])


def compare(args) -> int:
    """Prefill and decode throughput of a model of the named design and of a Qwen3 model of the same layer sizes
    (random weights, `--layers` layers each, default 4), then the design's kernels one by one beside their like
    kernels.  One JSON line per model and per kernel."""
    import numpy as np
    import torch
    from xinfer_b200 import measure
    from xinfer_b200.engine.runner import ModelRunner, StepInput
    pk = peaks()
    z = COMPARE_SIZES[args.size]
    L, V, B, ctx_len = args.layers or 4, 32000, args.batch, 2048
    qwen3 = dict(CONFIG, vocab_size=V, hidden_size=z["hidden"], intermediate_size=z["intermediate"], num_hidden_layers=L,
                 num_attention_heads=z["heads"], num_key_value_heads=z["kv_heads"], head_dim=z["head_dim"])
    if args.compare == "gulipel":       # its closest model is the other one with two mixers side by side
        models = {"Gulipel": gulipel_config(z, L, V, ctx_len + 128), "Tidarax": tidarax_config(z, L, V)}
    elif args.compare == "mikutar":     # its closest model is the other one with gated window attention and a float32 stream
        models = {"Mikutar": mikutar_config(z, L, V), "Mikutar, first layers twice": mikutar_config(z, L, V, loop=True),
                  "Dufitar": dufitar_config(z, LATENT_SIZES[args.size], L, V)}
    elif args.compare == "dalalix":     # gated attention and experts as in Mikutar, a matrix state beside attention as in Gulipel
        models = {"Dalalix": dalalix_config(z, L, V), "Mikutar": mikutar_config(z, L, V), "Gulipel": gulipel_config(z, L, V, ctx_len + 128)}
    elif args.compare == "napuzen":     # latent attention as in Dufitar, a recurrence with a matrix state as in Gulipel
        models = {"Napuzen": napuzen_config(z, LATENT_SIZES[args.size], L, V), "Dufitar": dufitar_config(z, LATENT_SIZES[args.size], L, V),
                  "Gulipel": gulipel_config(z, L, V, ctx_len + 128)}
    elif args.compare == "tidarax":
        models = {"Tidarax": tidarax_config(z, L, V), "Qwen3": qwen3}
    else:
        models = {"Dufitar": dufitar_config(z, LATENT_SIZES[args.size], L, V), "Qwen3": qwen3}
    rng = np.random.default_rng(0)
    for name, cfg in models.items():
        pages = (ctx_len + 64 + PAGE - 1) // PAGE + 1
        runner = ModelRunner.random(cfg, seed=0, dtype="bfloat16", block_size=PAGE, num_blocks=(B + 1) * pages, max_num_seqs=B + 1,
                                    max_model_len=ctx_len + 128)
        pre = []
        for i in range(5):
            s = runner.open_request()
            ids = rng.integers(0, V, size=PREFILL_TOKENS)
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            logits = runner.step([StepInput(s, ids, [PREFILL_TOKENS - 1])])
            e1.record()
            torch.cuda.synchronize()
            if i == 0:
                check_finite(logits, f"the first prefill of {name}")
            if i >= 2:
                pre.append(e0.elapsed_time(e1))
            runner.close_request(s)
        slots = [runner.open_request() for _ in range(B)]
        for s in slots:
            runner.step([StepInput(s, rng.integers(0, V, size=ctx_len - 64), [])])
        steps, warm = 32, 8 + SETTLE
        toks = rng.integers(0, V, size=(steps + warm, B))
        for i in range(warm):
            runner.step([StepInput(s, toks[i, j:j + 1], [0]) for j, s in enumerate(slots)], allow_graph=not args.no_graph)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for i in range(warm, warm + steps):
            logits = runner.step([StepInput(s, toks[i, j:j + 1], [0]) for j, s in enumerate(slots)], allow_graph=not args.no_graph)
        e1.record()
        torch.cuda.synchronize()
        runner.check_errors()
        check_finite(logits, f"the last decode step of {name}")
        ms = e0.elapsed_time(e1) / steps
        print(json.dumps({"model": name, "size": args.size, "layers": L, "weight_gb": round(runner.model.weight_bytes() / 1e9, 3),
                          "prefill_tokens": PREFILL_TOKENS, "prefill_ms": round(min(pre), 3),
                          "prefill_tok_s": round(PREFILL_TOKENS / (min(pre) / 1e3), 1), "decode_batch": B,
                          "decode_context": ctx_len, "decode_ms_per_step": round(ms, 4), "decode_tok_s": round(B / (ms / 1e3), 1),
                          "launches_per_decode_step": runner.last_launches, "cuda_graph": runner.last_used_graph,
                          "dtype": "bf16", "data": "synthetic (random weights, seeded uniform token ids)"}), flush=True)
        del runner
        torch.cuda.empty_cache()
    if args.compare == "mikutar":
        records = measure.mikutar_kernels(hidden=z["hidden"], heads=z["heads"], kv_heads=z["kv_heads"], head_dim=z["head_dim"],
                                          intermediate=z["intermediate"], experts=z["experts"], expert_ff=z["expert_ff"],
                                          top=z["top"], hbm_gbs=pk["hbm_gbs"], peak_tflops=pk["bf16_tflops"])
    elif args.compare == "dalalix":
        records = measure.dalalix_kernels(hidden=z["hidden"], heads=z["heads"], kv_heads=z["kv_heads"], head_dim=z["head_dim"],
                                          experts=z["experts"], expert_ff=z["expert_ff"], top=z["top"], hbm_gbs=pk["hbm_gbs"],
                                          peak_tflops=pk["bf16_tflops"])
    elif args.compare == "napuzen":
        lat = LATENT_SIZES[args.size]
        records = measure.napuzen_kernels(hidden=z["hidden"], heads=z["heads"], head_dim=z["head_dim"], kv_rank=lat["kv_rank"],
                                          rot_dim=lat["rot_dim"], q_rank=3 * lat["kv_rank"], experts=z["experts"],
                                          expert_ff=z["expert_ff"], top=z["top"], hbm_gbs=pk["hbm_gbs"], peak_tflops=pk["bf16_tflops"])
    elif args.compare == "gulipel":
        records = measure.gulipel_kernels(hidden=z["hidden"], heads=z["heads"], kv_heads=z["kv_heads"], head_dim=z["head_dim"],
                                          intermediate=z["intermediate"], hbm_gbs=pk["hbm_gbs"], **gulipel_sizes(z))
    elif args.compare == "dufitar":
        lat = LATENT_SIZES[args.size]
        records = measure.dufitar_kernels(hidden=z["hidden"], heads=z["heads"], kv_heads=z["kv_heads"], head_dim=z["head_dim"],
                                          intermediate=z["intermediate"], kv_rank=lat["kv_rank"], rot_dim=lat["rot_dim"],
                                          hbm_gbs=pk["hbm_gbs"], peak_tflops=pk["bf16_tflops"])
    else:
        records = measure.tidarax_kernels(hidden=z["hidden"], heads=z["heads"], kv_heads=z["kv_heads"], head_dim=z["head_dim"],
                                          intermediate=z["intermediate"], rec_width=z["hidden"], experts=z["experts"],
                                          expert_ff=z["expert_ff"], top=z["top"], hbm_gbs=pk["hbm_gbs"],
                                          peak_tflops=pk["bf16_tflops"])
    for rec in records:
        print(json.dumps(dict(rec, size=args.size)), flush=True)
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--shape", default="8b", choices=sorted(SHAPES),
                    help="layer sizes: the headline Qwen3-8B shape (default) or the 0.6B / 32B shapes")
    ap.add_argument("--layers", type=int, default=0,
                    help="run fewer layers than the configuration has (reported in config)")
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=CONTEXT)
    ap.add_argument("--no-points", action="store_true", help="skip the batch 1 / 64 points")
    ap.add_argument("--no-graph", action="store_true")
    ap.add_argument("--workload", default="steps", choices=["steps", "mixed"],
                    help="'mixed': 64 requests of 16..2,048 prompt tokens under continuous batching, instead of the step benchmark")
    ap.add_argument("--requests", type=int, default=64, help="requests of the mixed workload")
    ap.add_argument("--ablate", action="store_true",
                    help="instead of the step benchmark: a decode step with one kind of kernel left out at a time (what each kind costs in the chain)")
    ap.add_argument("--attn", default="", metavar="HEADS,KV_HEADS,HEAD_DIM[,PAGE_SIZE]",
                    help="with --kernels: the attention kernels alone at this head layout, over short and long contexts")
    ap.add_argument("--case", default="", metavar="decode:BATCHxCONTEXT | prefill:CACHED+NEW",
                    help="with --kernels --attn: this one case instead of the standard ones")
    ap.add_argument("--compare", default="", choices=["", "tidarax", "dufitar", "gulipel", "mikutar", "napuzen", "dalalix"],
                    help="instead of the step benchmark: prefill and decode throughput of this design beside its closest model "
                         "(Qwen3; for gulipel, Tidarax; for mikutar, Dufitar; for napuzen, Dufitar and Gulipel; for dalalix, Mikutar and Gulipel) at equal layer sizes, and its kernels beside their like kernels; one JSON line each")
    ap.add_argument("--size", default="4k", choices=sorted(COMPARE_SIZES), help="layer sizes of --compare")
    ap.add_argument("--kernels", action="store_true",
                    help="instead of the step benchmark, time single kernels at serving sizes: one JSON line each")
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm()
    if args.gpus != 1:
        print("bench.py: this engine runs on one GPU; --gpus must be 1")
        return 2
    steps, warmup = max(args.steps, 1), max(args.warmup, 3)
    if args.compare:
        return compare(args)
    if args.ablate:
        from xinfer_b200 import measure
        for rec in measure.decode_ablation(dict(CONFIG, **SHAPES[args.shape]), layers=args.layers or 12):
            print(json.dumps(rec), flush=True)
        return 0
    if args.kernels and args.attn:
        # the attention kernels alone at another head layout: HEADS,KV_HEADS,HEAD_DIM[,PAGE_SIZE]
        from xinfer_b200 import measure
        pk = peaks()
        sizes = [int(x) for x in args.attn.split(",")]
        lay = dict(heads=sizes[0], kv_heads=sizes[1], head_dim=sizes[2], page_size=sizes[3] if len(sizes) > 3 else PAGE)
        decode_cases, prefill_cases = ((1, 4096), (8, 4096), (64, 2048), (4, 65536), (16, 512)), ((0, 512), (0, 2048), (0, 8192), (30000, 2048))
        if args.case:      # one case alone (its first launch is a plain one: what a profiler is pointed at)
            kind, _, size = args.case.partition(":")
            if kind == "decode":
                decode_cases, prefill_cases = (tuple(int(x) for x in size.split("x")),), ()
            elif kind == "prefill":
                decode_cases, prefill_cases = (), (tuple(int(x) for x in size.split("+")),)
            else:
                raise SystemExit("bench.py: --case is decode:BATCHxCONTEXT or prefill:CACHED+NEW")
        for rec in (measure.decode_attention(decode_cases, hbm_gbs=pk["hbm_gbs"], **lay)
                    + measure.prefill_attention(prefill_cases, peak_tflops=pk["bf16_tflops"], **lay)):
            print(json.dumps(dict(rec, **lay)), flush=True)
        return 0
    if args.kernels:
        from xinfer_b200 import measure
        pk = peaks()
        for rec in (measure.decode_gemms(hbm_gbs=pk["hbm_gbs"]) + measure.decode_attention(hbm_gbs=pk["hbm_gbs"])
                    + measure.prefill_attention(peak_tflops=pk["bf16_tflops"]) + measure.prefill_elementwise(hbm_gbs=pk["hbm_gbs"])
                    + measure.sampling()):
            print(json.dumps(rec), flush=True)
        return 0

    import numpy as np
    import torch
    from xinfer_b200 import kernels
    from xinfer_b200.config import EngineConfig
    from xinfer_b200.engine.llm import Engine
    from xinfer_b200.engine.runner import ModelRunner, StepInput
    from xinfer_b200.sampling import SamplingParams

    pk = peaks()
    full = dict(CONFIG, **SHAPES[args.shape])
    cfg = dict(full, num_hidden_layers=args.layers or full["num_hidden_layers"])
    if args.workload == "mixed":
        return mixed_workload(args, cfg, full, pk)
    max_b = args.batch if args.no_points else max(args.batch, 64)
    if args.context < 256:
        raise SystemExit("bench.py: --context must be at least 256")
    longest = max(args.context, PREFILL_TOKENS + 256)     # the prefill measurement and the reference's decode setting need their room
    pages_per_req = (longest + PAGE - 1) // PAGE + 1
    t_load = time.time()
    runner = ModelRunner.random(cfg, seed=0, dtype="bfloat16", block_size=PAGE, num_blocks=max_b * pages_per_req,
                                max_num_seqs=max_b, max_model_len=longest + 64)
    torch.cuda.synchronize()
    load_s = time.time() - t_load
    rng = np.random.default_rng(0)
    V = cfg["vocab_size"]
    use_graph = not args.no_graph

    def fill(batch: int, ctx: int):
        """Open `batch` requests and prefill each to `ctx` tokens through the step function."""
        slots = [runner.open_request() for _ in range(batch)]
        chunk = 4096
        for s in slots:
            at = 0
            while at < ctx:
                n = min(chunk, ctx - at)
                runner.step([StepInput(s, rng.integers(0, V, size=n), [])])
                at += n
        runner.check_errors()
        return slots

    def decode_device(slots, n_steps: int, n_warm: int):
        """K decode steps, kernel time only: token ids come from the host each step, no read-back."""
        n_warm += SETTLE   # the prefill before leaves the device at its power cap: untimed steps until the clocks are back
        toks = rng.integers(0, V, size=(n_steps + n_warm, len(slots)))
        for i in range(n_warm):
            runner.step([StepInput(s, toks[i, j:j + 1], [0]) for j, s in enumerate(slots)], allow_graph=use_graph)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        launches = 0
        t0 = time.time()
        e0.record()
        for i in range(n_warm, n_warm + n_steps):
            runner.step([StepInput(s, toks[i, j:j + 1], [0]) for j, s in enumerate(slots)], allow_graph=use_graph)
            launches += runner.last_launches
        e1.record()
        torch.cuda.synchronize()
        t1 = time.time()
        runner.check_errors()
        return e0.elapsed_time(e1) / n_steps, launches, (t0, t1)

    def close(slots):
        for s in slots:
            runner.close_request(s)

    clocks = ClockSampler()
    clocks.start()

    # ---- prefill: one step of 2,048 prompt tokens ------------------------------------------------------
    pre_ms = []
    for i in range(3 + 3):
        s = runner.open_request()
        ids = rng.integers(0, V, size=PREFILL_TOKENS)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        logits = runner.step([StepInput(s, ids, [PREFILL_TOKENS - 1])])
        e1.record()
        torch.cuda.synchronize()
        if i == 0:
            absmax_prefill = check_finite(logits, "the first prefill")
        if i >= 3:
            pre_ms.append(e0.elapsed_time(e1))
        runner.close_request(s)
    runner.check_errors()
    pre = min(pre_ms)
    L, H, I = cfg["num_hidden_layers"], cfg["hidden_size"], cfg["intermediate_size"]
    nh, nkv, d = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    layer_params = H * (nh + 2 * nkv) * d + nh * d * H + 3 * H * I
    T = PREFILL_TOKENS
    flops = 2.0 * T * layer_params * L + 2.0 * V * H + L * 4.0 * nh * d * (T * (T + 1) / 2)
    prefill = {"value": round(T / (pre / 1e3), 1), "tokens": T, "ms": round(pre, 3),
               "frac": round(flops / (pre / 1e3) / (pk["bf16_tflops"] * 1e12), 4),
               "frac_nominal": round(flops / (pre / 1e3) / (NOMINAL_BF16_TFLOPS * 1e12), 4)}

    # ---- decode at the headline batch --------------------------------------------------------------------
    B = args.batch
    ctx0 = args.context - steps - warmup - SETTLE - 2
    if ctx0 < 16:
        raise SystemExit(f"bench.py: --steps {steps} with --warmup {warmup} does not fit a context of {args.context} "
                         f"(the timed steps end at the context length): give a larger --context or fewer steps")
    slots = fill(B, ctx0)
    ms, launches, (t0, t1) = decode_device(slots, steps, warmup)
    ck = clocks.summary(t0, t1)
    value = B / (ms / 1e3)
    weight_bytes = (layer_params * L + V * H) * 2 + (2 * L + 1) * H * 4 + L * 2 * d * 4
    ctx_mid = ctx0 + warmup + SETTLE + steps / 2
    kv_bytes = runner.kv_bytes_per_token * ctx_mid * B
    achieved = (weight_bytes + kv_bytes) / (ms / 1e3) / 1e9
    roofline = {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                "frac": round(achieved / pk["hbm_gbs"], 4), "frac_nominal": round(achieved / NOMINAL_HBM_GBS, 4)}
    absmax_decode = check_finite(runner.step([StepInput(s, rng.integers(0, V, size=1), [0]) for s in slots],
                                             allow_graph=use_graph), "the last decode step")
    close(slots)

    # ---- the same through the Python entry point ----------------------------------------------------------
    econfig = EngineConfig(weight_path="(random)", block_size=PAGE, max_num_seqs=max_b, max_num_batched_tokens=8192,
                           prefill_chunk_size=4096, max_model_len=longest + 64, disable_cuda_graph=not use_graph)
    engine = Engine(econfig, "bf16", runner=runner)
    n_e2e = min(steps, 64)
    # prompts are prefilled two per step, so requests start decoding a few steps apart: leave room
    # for that in the context, and let no request finish inside the timed region
    # the prompts' prefill leaves the device at its power cap for some tens of milliseconds: decode steps
    # run untimed until the clocks have come back
    e2e_warmup = warmup + SETTLE
    margin = B // 2 + 8
    prompt_len = args.context - n_e2e - e2e_warmup - margin - 8     # prompt + max_tokens stays inside a request's pages
    sp = SamplingParams(temperature=0.0, max_tokens=n_e2e + e2e_warmup + margin, ignore_eos=True)
    for _ in range(B):
        engine.add_request(rng.integers(0, V, size=prompt_len).tolist(), sp)
    while any(engine.scheduler.output(i) == [] for i in list(engine._live)):   # prompts, first tokens
        engine.step()
    for _ in range(e2e_warmup):
        engine.step()
    # The clock runs from one step's tokens reaching the host to those of the n-th step after it.  The
    # engine queues the next step before it waits for the current one, so the device is never drained
    # here: a synchronisation at the start would let the first timed call find its step already done.
    tw0 = time.time()
    done_before = engine.stats["decoded_tokens"]
    h2d = 0
    for _ in range(n_e2e):
        engine.step()   # returns when this step's tokens are on the host (the next step is already queued)
        h2d += runner.assembler.h2d_bytes + B * kernels.SAMPLE_PARAMS.itemsize
    tw1 = time.time()
    torch.cuda.synchronize()
    e2e_tokens = engine.stats["decoded_tokens"] - done_before
    e2e = {"value": round(e2e_tokens / (tw1 - tw0), 1), "unit": "tokens/s", "h2d_bytes_per_step": h2d // n_e2e,
           "d2h_bytes_per_step": B * 4 + 4}
    for seq_id in list(engine._live):   # the timed steps are done: drop what is still running
        engine.scheduler.abort(seq_id)
    while engine.has_work():
        engine.step()
    for seq_id in engine.scheduler.drain_finished():
        engine._finish(seq_id)

    # ---- batch 1 and 64 -----------------------------------------------------------------------------------
    points = {}
    if not args.no_points:
        for b in (1, 64):
            k = min(steps, 32)
            sl = fill(b, args.context - k - warmup - SETTLE - 2)
            m, _, _ = decode_device(sl, k, warmup)
            points[f"decode_b{b}"] = round(b / (m / 1e3), 1)
            close(sl)
        # the reference configuration's own decode setting: a 2,048-token prompt, then 256 decoded tokens
        for b in (1, 8, 64):
            sl = fill(b, PREFILL_TOKENS - warmup - SETTLE)
            m, _, _ = decode_device(sl, 256, warmup)
            points[f"baseline_b{b}"] = round(b / (m / 1e3), 1)
            close(sl)
    clocks.stop()

    out = {
        "metric": f"decode tok/s at batch {B} (Qwen3-{args.shape.upper()} shape, context {args.context})", "value": round(value, 1), "unit": "tokens/s",
        "n_gpus": 1, "steps": steps, "warmup": warmup, "ms_per_step": round(ms, 4), "higher_is_better": True,
        "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random weights, seeded uniform token ids)",
        "impl": "ours",
        "config": {"model": f"Qwen3-{args.shape.upper()} shape", "layers": cfg["num_hidden_layers"], "layers_of_config": full["num_hidden_layers"],
                   "hidden": H, "heads": nh, "kv_heads": nkv, "head_dim": d, "intermediate": I, "vocab": V,
                   "global_batch": B, "seq_len": args.context, "page_size": PAGE, "parallelism": "1 GPU",
                   "cuda_graph": use_graph, "l2": "inputs larger than L2 (weights read every step)",
                   "peaks": pk["source"], "settle_steps": SETTLE,
                   "logit_absmax_prefill": absmax_prefill, "logit_absmax_decode": absmax_decode},
        "clocks": ck, "e2e": e2e, "gpu_launches": int(launches), "prefill": prefill, "roofline": roofline, "points": points,
    }
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
