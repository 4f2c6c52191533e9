#!/usr/bin/env python3
"""Decode and prefill throughput of the Qwen3-1.7B shape with random weights on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--impl ours|reference]

Prints ONE JSON line.  ``value`` is decoded tokens a second at the default batch (8), timed on
the device with CUDA events around K decode steps of the step function plus the sampler (the
weights alone, 3.4 GB, exceed the 126 MB L2, so nothing is flushed between steps); the K-step
region is repeated until about a second has been timed and the median is reported.  ``e2e`` is
the same through the Python entry point (``Engine.step``: host token ids in through pinned
memory, sampled ids back to the host, every step) by wall clock, with the bytes each step really
copied; ``prefill`` is one request of 2,048 tokens in one step; ``points`` holds decode at batch
1 and 64 (``points_e2e`` the same end to end); ``roofline`` divides the bytes a decode step has
to read (every weight once, and the cache of the live requests) by its time.  A "step" is one
decode step.

Other workloads of the same engine, one JSON line each (not part of the default run):

    python bench.py --workload serving-8b    # Qwen3-8B shape: 64 requests, prompts U[128, 2048], 512-token portions, 256 tokens each
    python bench.py --workload qwen3-32b     # Qwen3-32B shape: 2,048-token prefill, decode at batch 1 and 8 to 4,096, cache from free memory
    python bench.py --workload fadosun [--breakdown]   # Fadosun beside Qwen3 at equal width, feed-forward and layers
    python bench.py --workload zufusun [--breakdown]   # Zufusun (two of eight experts a token) beside Qwen3 likewise
    python bench.py --workload fomanex [--breakdown]   # Fomanex beside Zufusun (its closest relative) and Qwen3 likewise
    python bench.py --workload pepapel [--breakdown]   # Pepapel beside Zufusun, Fadosun (its closest relatives) and Qwen3 likewise
    python bench.py --workload filanex [--breakdown]   # Filanex beside Pepapel (its closest relative) and Qwen3 likewise
    python bench.py --workload malusun [--breakdown]   # Malusun beside Zufusun and Fadosun (its closest relatives) and Qwen3 likewise
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

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_1P7B = dict(architectures=["Qwen3ForCausalLM"], model_type="qwen3", vocab_size=151936, hidden_size=2048,
                  intermediate_size=6144, num_hidden_layers=28, num_attention_heads=16, num_key_value_heads=8,
                  head_dim=128, rope_theta=1000000.0, rms_norm_eps=1e-6, tie_word_embeddings=True,
                  max_position_embeddings=40960)
QWEN3_8B = dict(QWEN3_1P7B, hidden_size=4096, intermediate_size=12288, num_hidden_layers=36, num_attention_heads=32,
                num_key_value_heads=8, tie_word_embeddings=False)
QWEN3_32B = dict(QWEN3_1P7B, hidden_size=5120, intermediate_size=25600, num_hidden_layers=64, num_attention_heads=64,
                 num_key_value_heads=8, tie_word_embeddings=False)
CONTEXT = 4096          # decode runs up to this many positions
DECODE_FROM = 3072      # the timed decode steps start here (the middle of 2,048 -> 4,096)
PREFILL_TOKENS = 2048
PAGE_TOKENS = 64          # the engine's default; the reference's block size is 16 (--page-tokens 16: a few per cent slower, more TMA boxes a tile)
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0, "source": "fallback"}


def peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(p):
        try:
            with open(p) as f:
                d = json.load(f)
            out = dict(FALLBACK_PEAKS)
            for k in ("hbm_gbs", "bf16_tflops", "bf16_tflops_sustained"):
                if isinstance(d.get(k), (int, float)) and d[k] > 0:
                    out[k] = float(d[k])
            out["source"] = "measured"
            return out
        except (OSError, ValueError):
            pass
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples nvidia-smi clocks and throttle reasons while the timed region runs."""

    FIELDS = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.proc, self.lines = None, []

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits",
                                          "-lms", "100"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=lambda: self.lines.extend(self.proc.stdout), daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def __exit__(self, *a):
        if self.proc:
            time.sleep(0.15)
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()
            self.thread.join(timeout=2)

    def summary(self):
        sm, mx, reasons = [], 0, set()
        for ln in self.lines:
            f = [x.strip() for x in ln.split(",")]
            if len(f) < 6:
                continue
            try:
                sm.append(int(f[0]))
                mx = max(mx, int(f[1]))
            except ValueError:
                continue
            for name, v in zip(("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"), f[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(name)
        return {"sm_mhz": int(statistics.median(sm)) if sm else None, "sm_max_mhz": mx or None,
                "reasons": sorted(reasons), "samples": len(sm)}


def model_bytes_and_flops(cfg, n_layers):
    """Bytes of weights a decode step reads once (bf16) and the flops of a T-token causal prefill."""
    H, I, V, D = cfg.hidden_size, cfg.intermediate_size, cfg.vocab_size, cfg.head_dim
    Q, KV = cfg.q_dim, cfg.kv_dim
    per_layer = H * (Q + 2 * KV) + Q * H + 3 * H * I
    weights = 2 * (n_layers * per_layer + V * H)                       # the head (tied: the embedding) is read once
    norms = 4 * (n_layers * (2 * H + 2 * D) + H)
    kv_per_token = 2 * n_layers * KV * 2                               # K and V, bf16

    def prefill_flops(T):
        linear = 2 * T * n_layers * per_layer + 2 * V * H              # head for one row
        attn = n_layers * cfg.num_attention_heads * 4 * D * (T * (T + 1) // 2)
        return linear + attn

    return weights + norms, kv_per_token, prefill_flops


def build_llm(cfg, n_layers, batch, seed=0, prefill_tokens=PREFILL_TOKENS):
    import ember_b200
    from ember_b200.config import Qwen3Config
    d = dict(cfg.to_json(), num_hidden_layers=n_layers, max_position_embeddings=max(cfg.max_position_embeddings, prefill_tokens))
    c = Qwen3Config.from_json(d)
    cap = max(batch * CONTEXT, prefill_tokens)
    return ember_b200.load_random(c, seed=seed, dtype="bfloat16", kv_cache_tokens=cap, page_tokens=PAGE_TOKENS,
                                  max_batch_tokens=max(prefill_tokens, 2048), max_seqs=max(batch, 1), prefill_chunk=2048)


def fill_cache(llm, batch, context):
    """Admits ``batch`` requests holding ``context`` tokens each without computing them: the pages
    are filled with random values (set-up only; a decode step's time does not depend on them)."""
    import torch
    r = llm.runner
    for t in r.storage._paged.values():
        for x in (t if isinstance(t, tuple) else (t,)):
            x.normal_(0.0, 0.5)
    ids = []
    for i in range(batch):
        rid = ("bench", i)
        assert r.admit(rid)
        assert r.cache.ensure(rid, context)
        r.cache.advance(rid, context)
        ids.append(rid)
    return ids


def time_decode(llm, batch, steps, warmup, context, min_total_ms=1000.0, max_steps=900):
    """K decode steps of the step function + sampler on the device, timed with CUDA events; the K-step region is
    repeated (at least 3 times, until ``min_total_ms`` has been timed, within ``max_steps`` positions) and the
    median taken.  Returns (ms per step, launches per step, repeats, mean context of the timed steps)."""
    import torch
    from ember_b200 import SamplingParams, StepEntry, ops
    from ember_b200.sampling import device as dsampler
    r = llm.runner
    ids = fill_cache(llm, batch, context)
    params = [SamplingParams(temperature=0.0)] * batch
    out = torch.empty(batch, dtype=torch.int32, device=r.device)
    vocab = r.spec.vocab_size

    def one(i):
        for rid in ids:
            assert r.reserve(rid, 1)
        entries = [StepEntry(rid, [(1000 + 7 * i + j) % vocab], (0,)) for j, rid in enumerate(ids)]
        logits = r.step(entries)
        dsampler.sample(logits, params, [context + i] * batch, out=out)

    def region(first):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        for i in range(steps):
            one(first + i)
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1) / steps

    for i in range(warmup):
        one(i)
    torch.cuda.synchronize()
    n0 = ops.launch_count()
    times = [region(warmup)]
    launches = (ops.launch_count() - n0) / steps
    done = warmup + steps
    while done + steps <= max_steps and (len(times) < 3 or sum(times) * steps < min_total_ms):
        times.append(region(done))
        done += steps
    r.check_device()
    for rid in ids:
        r.release(rid)
    mean_context = context + warmup + (done - warmup) / 2.0
    return statistics.median(times), launches, len(times), mean_context


def time_e2e(llm, batch, steps, warmup, context, min_total_ms=500.0, max_steps=900):
    """The same decode through Engine.step: host ids in (pinned staging), sampled ids out, each step, by wall
    clock; K-step regions repeated and the median taken.  Also the bytes a step copied each way, counted where
    the copies are made (``ember_b200.transfers``)."""
    import torch
    from ember_b200 import Request, SamplingParams, transfers
    eng = llm.engine
    vocab = llm.runner.spec.vocab_size
    # requests whose prompts are already cached: prefill them for real through the engine
    import random
    rng = random.Random(1234)
    seqs = [eng.submit(Request(prompt=[rng.randrange(1000, min(100000, vocab)) for _ in range(context)],
                               sampling=SamplingParams(temperature=0.0), max_tokens=CONTEXT - context - 8, ignore_eos=True))
            for _ in range(batch)]
    while not all(s.generated >= 1 for s in seqs):
        eng.step()
    for _ in range(warmup):
        eng.step()
    times, done = [], warmup
    h0, d0 = transfers.snapshot()
    while done + steps <= max_steps and (len(times) < 3 or sum(times) * steps < min_total_ms):
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        for _ in range(steps):
            eng.step()
        torch.cuda.synchronize()
        times.append((time.perf_counter() - t0) * 1000.0 / steps)
        done += steps
    h1, d1 = transfers.snapshot()
    n = steps * len(times)
    for s in seqs:
        s.cancelled = True
    eng.step()
    eng.drain()
    llm.runner.check_device()
    return statistics.median(times), (h1 - h0) // n, (d1 - d0) // n


def time_prefill(llm, tokens, reps, warmup):
    import torch
    from ember_b200 import StepEntry
    r = llm.runner
    vocab = r.spec.vocab_size
    import random
    rng = random.Random(4321)
    times = []
    for i in range(warmup + reps):
        rid = ("prefill", i)
        assert r.admit(rid) and r.reserve(rid, tokens)
        toks = [rng.randrange(1000, min(100000, vocab)) for _ in range(tokens)]
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        r.step([StepEntry(rid, toks, (tokens - 1,))])
        e1.record()
        torch.cuda.synchronize()
        if i >= warmup:
            times.append(e0.elapsed_time(e1))
        r.release(rid)
    r.check_device()
    return statistics.median(times)


def breakdown(cfg, n_layers, batch) -> int:
    """Per-kernel device time of decode steps and of a prefill step, kernels serialised (no programmatic
    dependent launch, no graphs), caches warm: what each kernel costs by itself inside a step."""
    os.environ["EMBER_PDL"] = "0"
    import torch
    from torch.profiler import ProfilerActivity, profile
    from ember_b200 import StepEntry
    import random
    llm = build_llm(cfg, n_layers, max(batch, 1))
    r = llm.runner
    r.cuda_graphs = False
    ids = fill_cache(llm, batch, DECODE_FROM)
    rng = random.Random(1)
    vocab = r.spec.vocab_size

    def decode():
        for rid in ids:
            assert r.reserve(rid, 1)
        r.step([StepEntry(rid, [rng.randrange(1000, min(100000, vocab))], (0,)) for rid in ids])

    def table(title, prof, steps):
        rows = [(e.key, e.self_device_time_total / steps, e.count // steps) for e in prof.key_averages()
                if e.self_device_time_total > 0]
        rows.sort(key=lambda x: -x[1])
        total = sum(x[1] for x in rows)
        print(f"{title}: {total / 1000:.3f} ms of kernels per step")
        for name, us, n in rows[:12]:
            print(f"  {us:9.1f} us {100 * us / total:5.1f} %  x{n:<4d} {name.split('(')[0][-60:]}")

    for _ in range(3):
        decode()
    torch.cuda.synchronize()
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        for _ in range(3):
            decode()
        torch.cuda.synchronize()
    table(f"decode step, batch {batch}, context {DECODE_FROM}, {n_layers} layers", prof, 3)
    for rid in ids:
        r.release(rid)
    toks = [rng.randrange(1000, min(100000, vocab)) for _ in range(PREFILL_TOKENS)]

    def prefill(i):
        rid = ("prefill", i)
        assert r.admit(rid) and r.reserve(rid, PREFILL_TOKENS)
        r.step([StepEntry(rid, toks, (PREFILL_TOKENS - 1,))])
        torch.cuda.synchronize()
        r.release(rid)

    for i in range(2):
        prefill(i)
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        prefill(2)
    table(f"prefill step, {PREFILL_TOKENS} tokens, {n_layers} layers", prof, 1)
    return 0


FADOSUN_LAYERS = [
    {"type": "channel_delta", "mixer": {"heads": 16, "kv_heads": 16, "dim": 128, "vdim": 128, "conv": 4, "decay_rank": 64,
                                        "gate_rank": 64}},
    {"type": "parallel", "mixer": {
        "left": {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 0.0884, "rot": {"dims": 64, "base": 1e6}},
        "right": {"heads": 32, "vdim": 64, "state": 128, "groups": 1, "norm_groups": 1, "conv": 4},
        "left_scale": 1.0, "right_scale": 1.0}},
    {"type": "mlstm", "mixer": {"heads": 8, "dim": 128, "vdim": 256, "gate_cap": 15.0}},
    {"type": "channel_delta", "mixer": {"heads": 16, "kv_heads": 16, "dim": 128, "vdim": 128, "conv": 4, "decay_rank": 64,
                                        "gate_rank": 64}},
]


ZUFUSUN_LAYERS = [
    {"type": "gla", "mixer": {"heads": 16, "dim": 128, "vdim": 128, "tau": 16.0, "decay_rank": 64}},
    {"type": "attention", "mixer": {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 0.0884,
                                    "mask": {"size": 512, "keep_first": 4}}},
    {"type": "latent_attention", "mixer": {"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": 768, "kv_rank": 512,
                                           "scale": 0.0722, "rot": {"dims": 64, "base": 1e6}}},
    {"type": "latent_attention", "mixer": {"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": 768, "kv_rank": 512,
                                           "scale": 0.0722, "rot": {"dims": 64, "base": 1e6}, "kv_from": -1}},
]


def workload_fadosun(args, pk) -> int:
    """Fadosun beside Qwen3 at equal width, feed-forward, vocabulary and number of layers (the 1.7B widths, 8 layers
    unless --layers says otherwise; random weights): prefill of 512 and 2,048 tokens and decode steps at batch 8 and 64
    from a context of 1,024; with --breakdown instead the device time per kernel of one 2,048-token prefill and of a
    decode step at batch 64 (kernels serialised: no programmatic dependent launch, no graphs)."""
    n_layers = args.layers or 8
    return beside_qwen3(args, pk, "fadosun", fadosun_config(n_layers), n_layers, {"fadosun_layers": [l["type"] for l in FADOSUN_LAYERS]})


def zufusun_config(n_layers):
    from ember_b200.config import ZufusunConfig
    width, ff, vocab = QWEN3_1P7B["hidden_size"], QWEN3_1P7B["intermediate_size"], QWEN3_1P7B["vocab_size"]
    mlp = {"kind": "moe", "expert": {"ff": ff // 2, "limit": 7.0}, "router": {"experts": 8, "top": 2}}
    layers = []
    for i in range(n_layers):
        l = json.loads(json.dumps(ZUFUSUN_LAYERS[i % 4]))
        if l["mixer"].get("kv_from") == -1:
            l["mixer"]["kv_from"] = i - 1              # the latent of the layer before it
        layers.append(dict(l, mlp=mlp))
    return ZufusunConfig.from_json({"architecture": "Zufusun", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": layers})


def workload_zufusun(args, pk) -> int:
    """Zufusun beside Qwen3 at equal width, vocabulary and number of layers (the 1.7B widths, 8 layers unless --layers
    says otherwise; random weights), its feed-forward eight experts of half Qwen3's feed-forward size of which a token
    uses two (the same products per token, four times the weights): the measurements of ``--workload fadosun``."""
    n_layers = args.layers or 8
    ff = QWEN3_1P7B["intermediate_size"]
    return beside_qwen3(args, pk, "zufusun", zufusun_config(n_layers), n_layers,
                        {"zufusun_layers": [l["type"] for l in ZUFUSUN_LAYERS], "experts": 8, "top": 2, "expert_ff": ff // 2})


FOMANEX_LAYERS = [
    {"type": "wkv", "mixer": {"heads": 16, "dim": 128, "decay_rank": 64}, "mlp": "dense"},
    {"type": "latent_attention", "mlp": "moe",
     "mixer": {"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 0.0722,
               "rot": {"dims": 64, "base": 1e6, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}},
]


def fomanex_config(runs):
    """(configuration, its dictionary) of ``runs`` layer runs: time mixing and latent attention alternate, a dense
    feed-forward of Qwen3's size after the one and eight experts of half that size, two a token, after the other; two
    copies of the residual stream; from 6 runs on, pairs of layers behind the first two are listed once and run twice."""
    from ember_b200.config import FomanexConfig
    looped = 2 * max((runs - 2) // 4, 0)               # layers listed once and run twice (whole wkv + latent pairs)
    listed = runs - looped
    width, ff, vocab = QWEN3_1P7B["hidden_size"], QWEN3_1P7B["intermediate_size"], QWEN3_1P7B["vocab_size"]
    mlps = {"dense": {"kind": "dense", "ff": ff},
            "moe": {"kind": "moe", "expert": {"ff": ff // 2}, "router": {"experts": 8, "top": 2, "scale": 2.5}}}
    layers = [dict(json.loads(json.dumps(FOMANEX_LAYERS[i % 2])), mlp=mlps[FOMANEX_LAYERS[i % 2]["mlp"]]) for i in range(listed)]
    cfg = {"architecture": "Fomanex", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 45.25},
           "residual_mult": 0.5, "streams": 2, "logit_scale": 0.25, "logit_softcap": 30.0, "layers": layers}
    if looped:
        cfg["loop"] = {"start": 2, "stop": 2 + looped, "times": 2}
    return FomanexConfig.from_json(cfg), cfg


def workload_fomanex(args, pk) -> int:
    """Fomanex beside Zufusun (the design whose latent attention, recurrence and experts are the like kernels) and
    Qwen3, all at the 1.7B width and vocabulary and with as many layer runs (8 unless --layers says otherwise; random
    weights); of 8 layer runs the third and fourth are one pair of layers run twice (a state and a cache per pass): the
    measurements of ``--workload fadosun``."""
    runs = args.layers or 8
    fcfg, cfg = fomanex_config(runs)
    return beside_qwen3(args, pk, "fomanex", fcfg, runs,
                        {"fomanex_layers": [l["type"] for l in FOMANEX_LAYERS], "listed_layers": len(cfg["layers"]), "loop": cfg.get("loop"),
                         "streams": 2, "experts": 8, "top": 2, "expert_ff": QWEN3_1P7B["intermediate_size"] // 2},
                        others=[("zufusun", zufusun_config(runs))])


def fadosun_config(n_layers):
    from ember_b200.config import FadosunConfig
    width, ff, vocab = QWEN3_1P7B["hidden_size"], QWEN3_1P7B["intermediate_size"], QWEN3_1P7B["vocab_size"]
    return FadosunConfig.from_json({"architecture": "Fadosun", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
                                    "layers": [dict(FADOSUN_LAYERS[i % 4], mlp={"kind": "dense", "ff": ff}) for i in range(n_layers)]})


PEPAPEL_LAYERS = [
    {"type": "parallel", "mixer": {
        "left": {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 0.0884, "conv": 4, "mask": {"size": 512},
                 "rot": {"dims": 64, "base": 1e6, "scaling": {"factor": 4.0}}},
        "right": {"heads": 16, "kv_heads": 16, "dim": 128, "vdim": 128, "conv": 4}}},
    {"type": "attention", "mixer": {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 0.0884, "softcap": 30.0,
                                    "q_temp": {"coef": 0.3, "every": 1024}}},
]


def pepapel_config(n_layers):
    """``n_layers`` layers: three parallel layers (attention inside chunks of 512 beside a delta rule of 16 heads of
    128 x 128) and one attention layer over all keys, in turn; the first layer's feed-forward is dense and of Qwen3's size,
    the others' eight experts of half that size plus two identity experts, two a token, from three of five groups."""
    from ember_b200.config import PepapelConfig
    width, ff, vocab = QWEN3_1P7B["hidden_size"], QWEN3_1P7B["intermediate_size"], QWEN3_1P7B["vocab_size"]
    moe = {"kind": "moe", "expert": {"ff": ff // 2}, "router": {"experts": 8, "top": 2, "identity": 2, "groups": {"count": 5, "keep": 3}}}
    layers = [dict(json.loads(json.dumps(PEPAPEL_LAYERS[0 if i % 4 < 3 else 1])), mlp=moe if i else {"kind": "dense", "ff": ff, "limit": 7.0})
              for i in range(n_layers)]
    return PepapelConfig.from_json({"architecture": "Pepapel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
                                    "embedding": {"scale": 45.25}, "postln_alpha": 2.0, "layers": layers})


def workload_pepapel(args, pk) -> int:
    """Pepapel beside Zufusun (whose attention and experts are the like kernels), Fadosun (whose delta rule and parallel
    layer are) and Qwen3, all at the 1.7B width and vocabulary and with as many layers (8 unless --layers says otherwise;
    random weights): the measurements of ``--workload fadosun``."""
    n_layers = args.layers or 8
    return beside_qwen3(args, pk, "pepapel", pepapel_config(n_layers), n_layers,
                        {"pepapel_layers": ["parallel", "parallel", "parallel", "attention"], "experts": 8, "identity": 2, "top": 2,
                         "expert_ff": QWEN3_1P7B["intermediate_size"] // 2},
                        others=[("zufusun", zufusun_config(n_layers)), ("fadosun", fadosun_config(n_layers))])


def filanex_config(runs):
    """``runs`` layer runs (6 or more) from two fewer listed layers: dense and expert feed-forwards in turn, attention inside
    chunks of 2,048 (so that a decode step at a context of 1,024 reads as many keys as Qwen3's), 16 / 8 heads of 128, half
    of each rotated, capped scores, a gate per element; the third and fourth layer run twice."""
    from ember_b200.config import FilanexConfig
    width, ff, vocab = QWEN3_1P7B["hidden_size"], QWEN3_1P7B["intermediate_size"], QWEN3_1P7B["vocab_size"]
    mixer = {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 50.0, "mask": {"size": 2048},
             "rot": {"dims": 64, "base": 1e6, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    mlps = [{"kind": "dense", "ff": ff},
            {"kind": "moe", "expert": {"ff": ff // 2}, "router": {"experts": 8, "top": 2, "groups": {"count": 4, "keep": 2}}}]
    layers = [{"type": "attention", "mixer": mixer, "mlp": mlps[i % 2]} for i in range(runs - 2)]
    return FilanexConfig.from_json({"architecture": "Filanex", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
                                    "embedding": {"bigram": {"buckets": 131071, "mul_prev": 7919, "mul_cur": 104729}},
                                    "loop": {"start": 2, "stop": 4, "times": 2}, "layers": layers})


def workload_filanex(args, pk) -> int:
    """Filanex beside Pepapel (whose attention and experts are the like kernels) and Qwen3, all at the 1.7B width and
    vocabulary and with as many layer runs (8 unless --layers says otherwise; random weights): the measurements of
    ``--workload fadosun``."""
    runs = max(args.layers or 8, 6)
    return beside_qwen3(args, pk, "filanex", filanex_config(runs), runs,
                        {"filanex_layers_listed": runs - 2, "loop": "layers 2 and 3 twice", "chunk": 2048, "experts": 8, "top": 2,
                         "expert_ff": QWEN3_1P7B["intermediate_size"] // 2}, others=[("pepapel", pepapel_config(runs))])


MALUSUN_MIXERS = [
    ("mamba1", {"inner": 4096, "state": 16, "dt_rank": 128, "conv": 4}),
    ("attention", {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 0.0884, "mask": {"size": 1024},
                   "rot": {"dims": 64, "base": 1e6}, "v_mix": True}),
    ("mamba1", {"inner": 4096, "state": 16, "dt_rank": 128, "conv": 4}),
    ("attention_2", {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 0.0884, "mask": {"size": 1024}, "v_mix": True}),
]


def malusun_config(n_layers):
    """``n_layers`` layers: selective scans (4,096 channels of 16 states) and attention in windows of 1,024 (16/8 heads of 128;
    rotated, then with distance slopes and the fixed sink, all blending values) in turn; the first feed-forward is dense and of
    Qwen3's size, the others' one of eight experts of half that size a token and a shared one of that size."""
    from ember_b200.config import MalusunConfig
    width, ff, vocab = QWEN3_1P7B["hidden_size"], QWEN3_1P7B["intermediate_size"], QWEN3_1P7B["vocab_size"]
    moe = {"kind": "moe", "expert": {"ff": ff // 2}, "router": {"experts": 8, "top": 1}, "shared": {"ff": ff // 2}}
    layers = [{"type": MALUSUN_MIXERS[i % 4][0], "mixer": MALUSUN_MIXERS[i % 4][1], "mlp": moe if i else {"kind": "dense", "ff": ff}}
              for i in range(n_layers)]
    return MalusunConfig.from_json({"architecture": "Malusun", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
                                    "embedding": {"scale": 45.25}, "layers": layers})


def workload_malusun(args, pk) -> int:
    """Malusun beside Zufusun (whose windowed attention with a sink and experts are the like kernels), Fadosun (whose state
    space, convolution and layers between two norms are) and Qwen3, all at the 1.7B width and vocabulary and with as many
    layers (8 unless --layers says otherwise; random weights): the measurements of ``--workload fadosun``."""
    n_layers = args.layers or 8
    return beside_qwen3(args, pk, "malusun", malusun_config(n_layers), n_layers,
                        {"malusun_layers": [k for k, _ in MALUSUN_MIXERS], "window": 1024, "experts": 8, "top": 1, "shared": 1,
                         "expert_ff": QWEN3_1P7B["intermediate_size"] // 2},
                        others=[("zufusun", zufusun_config(n_layers)), ("fadosun", fadosun_config(n_layers))])


def beside_qwen3(args, pk, label, fcfg, n_layers, extra, others=()) -> int:
    """A design (``fcfg``) and Qwen3 at the 1.7B widths and ``n_layers`` layers, one after the other: prefill of 512 and
    2,048 tokens and decode steps at batch 8 and 64 from a context of 1,024, or with --breakdown the device time per
    kernel of one 2,048-token prefill and of a decode step at batch 64.  ``others``: (name, configuration) of further
    models of ``n_layers`` layer runs measured between the two."""
    import torch
    import ember_b200
    from ember_b200 import ops
    from ember_b200.config import Qwen3Config
    if args.breakdown:
        os.environ["EMBER_PDL"] = "0"          # kernels one after the other: each one's own time
    width, ff, vocab = QWEN3_1P7B["hidden_size"], QWEN3_1P7B["intermediate_size"], QWEN3_1P7B["vocab_size"]
    context, warmup = 1024, max(3, args.warmup)
    qcfg = Qwen3Config.from_json(dict(QWEN3_1P7B, num_hidden_layers=n_layers))

    def build(cfg, batch):
        return ember_b200.load_random(cfg, seed=0, dtype="bfloat16", kv_cache_tokens=max(batch * (context + 512), 2048),
                                      page_tokens=PAGE_TOKENS, max_batch_tokens=2048, max_seqs=max(batch, 1), prefill_chunk=2048)

    def kernel_table(llm, batch):
        """us per kernel name for one 2,048-token prefill and for a decode step at ``batch`` (kernels serialised)."""
        from torch.profiler import ProfilerActivity, profile
        from ember_b200 import StepEntry
        import random
        r = llm.runner
        r.cuda_graphs = False
        rng = random.Random(1)
        toks = [rng.randrange(1000, 100000) for _ in range(2048)]
        out = {}

        def prefill(i):
            rid = ("kp", i)
            assert r.admit(rid) and r.reserve(rid, 2048)
            r.step([StepEntry(rid, toks, (2047,))])
            torch.cuda.synchronize()
            r.release(rid)

        def rows(prof, steps):
            t = {}
            for e in prof.key_averages():
                if e.self_device_time_total > 0:
                    name = e.key.split("(")[0].split("<")[0].split("::")[-1][-48:]
                    t[name] = t.get(name, 0.0) + e.self_device_time_total / steps
            return {k: round(v, 1) for k, v in sorted(t.items(), key=lambda x: -x[1])[:14]}

        for i in range(2):
            prefill(i)
        with profile(activities=[ProfilerActivity.CUDA]) as prof:
            prefill(2)
        out["prefill_2048_us"] = rows(prof, 1)
        ids = fill_cache(llm, batch, context)

        def decode():
            for rid in ids:
                assert r.reserve(rid, 1)
            r.step([StepEntry(rid, [rng.randrange(1000, 100000)], (0,)) for rid in ids])

        for _ in range(3):
            decode()
        torch.cuda.synchronize()
        with profile(activities=[ProfilerActivity.CUDA]) as prof:
            for _ in range(3):
                decode()
            torch.cuda.synchronize()
        out[f"decode_b{batch}_us"] = rows(prof, 3)
        for rid in ids:
            r.release(rid)
        return out

    result = {"workload": label, "layers": n_layers, "width": width, "ff": ff, "vocab": vocab, "dtype": "bf16",
              "data": "synthetic (random weights from a seed, random token ids)", "decode_from": context,
              "page_tokens": PAGE_TOKENS, "peaks": pk["source"]}
    result.update(extra)
    with ClockSampler() as clocks:
        for name, cfg in ((label, fcfg),) + tuple(others) + (("qwen3", qcfg),):
            res = {}
            llm = build(cfg, 64)
            if args.breakdown:
                res["kernels"] = kernel_table(llm, 64)
            for n_tok in (() if args.breakdown else (512, 2048)):
                pms = time_prefill(llm, n_tok, reps=3, warmup=2)
                res[f"prefill_{n_tok}"] = {"ms": round(pms, 3), "tokens_per_s": round(n_tok / (pms * 1e-3), 1)}
            for batch in (() if args.breakdown else (8, 64)):
                steps = max(8, args.steps // (1 if batch == 8 else 2))
                ms, launches, _, _ = time_decode(llm, batch, steps, warmup, context, min_total_ms=300.0, max_steps=400)
                res[f"decode_b{batch}"] = {"ms_per_step": round(ms, 4), "tokens_per_s": round(batch * 1000.0 / ms, 1),
                                           "launches_per_step": round(launches, 1)}
            result[name] = res
            del llm
            torch.cuda.empty_cache()
    result["clocks"] = clocks.summary()
    result["gpu_launches"] = ops.launch_count()
    print(json.dumps(result))
    return 0


def workload_serving_8b(args, pk) -> int:
    """BASELINE's fourth configuration: the Qwen3-8B shape, 64 requests with random-id prompts of lengths uniform in
    [128, 2048], continuous batching with 512-token prompt portions, 256 decoded tokens each, through ``Engine``
    (host ids in, host ids out).  The cache is sized from the device's free memory."""
    import random
    import torch
    import ember_b200
    from ember_b200 import Request, SamplingParams
    from ember_b200.config import Qwen3Config
    cfg = Qwen3Config.from_json(dict(QWEN3_8B, num_hidden_layers=args.layers or QWEN3_8B["num_hidden_layers"]))
    n_layers = cfg.num_hidden_layers
    wbytes, kv_per_token, _ = model_bytes_and_flops(cfg, n_layers)
    n_req, gen, chunk = 64, 256, 512
    with ClockSampler() as clocks:
        llm = ember_b200.load_random(cfg, seed=0, dtype="bfloat16", kv_cache_tokens=0, page_tokens=PAGE_TOKENS,
                                     max_batch_tokens=2048, max_seqs=64, prefill_chunk=chunk, max_context=4096)
        eng, vocab = llm.engine, cfg.vocab_size
        rng = random.Random(1234)
        greedy = SamplingParams(temperature=0.0)

        def submit(n, lo, hi, ntok):
            return [eng.submit(Request(prompt=[rng.randrange(1000, min(100000, vocab)) for _ in range(rng.randint(lo, hi))],
                                       sampling=greedy, max_tokens=ntok, ignore_eos=True)) for _ in range(n)]

        def run(seqs, trace=None):
            sched = eng.scheduler
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            while any(s.finished is None for s in seqs):
                before = sched.stats.prompt_tokens + sched.stats.generated_tokens
                if not eng.step():
                    break
                if trace is not None:      # (tokens this commit accounted for, tokens cached by the running requests, how many run)
                    trace.append((sched.stats.prompt_tokens + sched.stats.generated_tokens - before,
                                  sum(q.computed for q in sched.running), len(sched.running)))
            eng.drain()
            torch.cuda.synchronize()
            return time.perf_counter() - t0

        run(submit(8, 128, 600, 8))                                   # warm-up: every kernel shape of the mix once
        s0 = eng.stats.steps
        seqs = submit(n_req, 128, 2048, gen)
        prompt_tokens = sum(q.prompt_len for q in seqs)
        trace = []
        dt = run(seqs, trace)
        llm.runner.check_device()
    steps = eng.stats.steps - s0
    generated = sum(len(q.output) for q in seqs)
    # the roofline of each step: the slower of reading (weights once + the running requests' cache) and computing
    # (2 flops per weight per token + attention over the cached tokens), summed over the steps
    H, D, nh = cfg.hidden_size, cfg.head_dim, cfg.num_attention_heads
    per_layer = H * (cfg.q_dim + 2 * cfg.kv_dim) + cfg.q_dim * H + 3 * H * cfg.intermediate_size
    bound_s, read_bytes, flops = 0.0, 0.0, 0.0
    for toks, live, running in trace:
        b = wbytes + live * kv_per_token
        # every token attends to about the mean cached length of the running requests
        f = 2.0 * max(toks, 1) * n_layers * per_layer + 2.0 * cfg.vocab_size * H * min(max(toks, 1), 64) \
            + 4.0 * n_layers * nh * D * (live / max(running, 1)) * max(toks, 1)
        bound_s += max(b / (pk["hbm_gbs"] * 1e9), f / (pk["bf16_tflops_sustained"] * 1e12))
        read_bytes += b
        flops += f
    out = {"metric": "continuous batching: generated tok/s, 64 requests, prompts U[128,2048], 512-token portions, 256 tokens each (Qwen3-8B shape)",
           "value": round(generated / dt, 1), "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": 1,
           "ms_per_step": round(dt * 1000.0 / max(steps, 1), 4), "higher_is_better": True, "dtype": "bf16", "impl": "ours",
           "data": "synthetic (random weights from a seed, random token ids)",
           "config": {"model": "Qwen3-8B shape", "requests": n_req, "prompt_tokens": prompt_tokens, "generated_tokens": generated,
                      "prefill_chunk": chunk, "max_batch_tokens": 2048, "max_seqs": 64, "layers": n_layers,
                      "layers_of_config": QWEN3_8B["num_hidden_layers"], "hidden": H, "intermediate": cfg.intermediate_size,
                      "heads": nh, "kv_heads": cfg.num_key_value_heads, "vocab": cfg.vocab_size, "page_tokens": PAGE_TOKENS,
                      "cache_tokens": llm.runner.cache.capacity_tokens(), "peaks": pk["source"]},
           "e2e": {"value": round(generated / dt, 1), "unit": "tokens/s", "total_tokens_per_s": round((generated + prompt_tokens) / dt, 1),
                   "seconds": round(dt, 3), "note": "this workload is end to end by construction (Engine.step, host ids in and out)"},
           "preemptions": eng.stats.preemptions,
           "roofline": {"bound": "per step, the slower of hbm and tensor", "frac": round(bound_s / dt, 4),
                        "hbm_frac": round(read_bytes / dt / 1e9 / pk["hbm_gbs"], 4),
                        "tensor_frac": round(flops / dt / 1e12 / pk["bf16_tflops_sustained"], 4)},
           "clocks": clocks.summary()}
    print(json.dumps(out))
    return 0


def workload_qwen3_32b(args, pk) -> int:
    """BASELINE's fifth configuration: the Qwen3-32B shape (65.5 GB of bf16 weights), a 2,048-token prefill, decode
    at batch 1 and 8 from context 3,072 towards 4,096, the cache sized from the memory the weights leave."""
    global CONTEXT
    import torch
    import ember_b200
    from ember_b200.config import Qwen3Config
    cfg = Qwen3Config.from_json(dict(QWEN3_32B, num_hidden_layers=args.layers or QWEN3_32B["num_hidden_layers"]))
    n_layers = cfg.num_hidden_layers
    wbytes, kv_per_token, prefill_flops = model_bytes_and_flops(cfg, n_layers)
    warmup = max(3, args.warmup)
    with ClockSampler() as clocks:
        t0 = time.perf_counter()
        llm = ember_b200.load_random(cfg, seed=0, dtype="bfloat16", kv_cache_tokens=0, page_tokens=PAGE_TOKENS,
                                     max_batch_tokens=2048, max_seqs=64, prefill_chunk=2048, gpu_memory=0.92)
        torch.cuda.synchronize()
        load_s = time.perf_counter() - t0
        r = llm.runner
        free, total = torch.cuda.mem_get_info()
        pms = time_prefill(llm, PREFILL_TOKENS, reps=3, warmup=2)
        points, fracs = {}, {}
        for b in (1, 8):
            ms, _, _, ctx = time_decode(llm, b, args.steps, warmup, DECODE_FROM, min_total_ms=1500.0,
                                        max_steps=CONTEXT - DECODE_FROM - 8)
            points[f"decode_b{b}"] = round(b * 1000.0 / ms, 1)
            fracs[f"decode_b{b}"] = round((wbytes + b * ctx * kv_per_token) / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)
            if b == 8:
                ms8, ctx8 = ms, ctx
    fl = prefill_flops(PREFILL_TOKENS)
    step_bytes = wbytes + 8 * ctx8 * kv_per_token
    out = {"metric": "decode tok/s at batch 1/8; prefill tok/s at 2,048 tokens (Qwen3-32B)", "value": points["decode_b8"],
           "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": warmup, "ms_per_step": round(ms8, 4),
           "higher_is_better": True, "dtype": "bf16", "impl": "ours",
           "data": "synthetic (random weights from a seed, random token ids)",
           "config": {"model": "Qwen3-32B shape", "global_batch": 8, "seq_len": CONTEXT, "decode_from": DECODE_FROM,
                      "layers": n_layers, "layers_of_config": QWEN3_32B["num_hidden_layers"], "hidden": cfg.hidden_size,
                      "intermediate": cfg.intermediate_size, "heads": cfg.num_attention_heads,
                      "kv_heads": cfg.num_key_value_heads, "vocab": cfg.vocab_size, "page_tokens": PAGE_TOKENS,
                      "gpu_memory": 0.92, "cache_tokens": r.cache.capacity_tokens(),
                      "cache_gib": round(r.storage.bytes() / 2**30, 1), "device_free_gib_after": round(free / 2**30, 1),
                      "load_seconds": round(load_s, 1), "peaks": pk["source"]},
           "roofline": {"bound": "hbm", "achieved": round(step_bytes / (ms8 * 1e-3) / 1e9, 1), "peak": pk["hbm_gbs"],
                        "unit": "GB/s", "frac": fracs["decode_b8"], "bytes_per_step": int(step_bytes)},
           "prefill": {"value": round(PREFILL_TOKENS / (pms * 1e-3), 1), "tokens": PREFILL_TOKENS, "ms": round(pms, 3),
                       "frac": round(fl / (pms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4), "tflops": round(fl / (pms * 1e-3) / 1e12, 1)},
           "points": points, "points_hbm_frac": fracs, "clocks": clocks.summary()}
    print(json.dumps(out))
    return 0


def main() -> int:
    global PAGE_TOKENS, CONTEXT, DECODE_FROM
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration has (named in config)")
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--skip-points", action="store_true", help="skip the batch 1 / 64 points and the prefill")
    ap.add_argument("--only-prefill", action="store_true", help="profiling aid: run just the 2,048-token prefill")
    ap.add_argument("--breakdown", action="store_true",
                    help="profiling aid: device time per kernel of three decode steps and one 2,048-token prefill step "
                         "(kernels serialised: EMBER_PDL=0 and no CUDA graphs are set by this flag)")
    ap.add_argument("--page-tokens", type=int, default=PAGE_TOKENS, choices=[16, 32, 64], help="tokens per cache page")
    ap.add_argument("--workload", default="default", choices=["default", "serving-8b", "qwen3-32b", "fadosun", "zufusun", "fomanex", "pepapel", "filanex", "malusun"],
                    help="default: the Qwen3-1.7B line; serving-8b and qwen3-32b are BASELINE's fourth "
                         "and fifth configurations; fadosun, zufusun, fomanex, pepapel, filanex, malusun: that design beside Qwen3 at equal sizes (with "
                         "--breakdown also per kernel); one JSON line each")
    ap.add_argument("--prefill-tokens", type=int, default=PREFILL_TOKENS,
                    help="with --only-prefill: another prompt length (the reported line stays at 2,048)")
    ap.add_argument("--decode-from", type=int, default=DECODE_FROM,
                    help="context length at which the timed decode steps start (other lengths than the default's "
                         "3,072: the cache is sized for it; `config` names it)")
    args = ap.parse_args()
    PAGE_TOKENS = args.page_tokens
    custom_context = None
    if args.decode_from != DECODE_FROM:
        custom_context = DECODE_FROM = max(1, args.decode_from)
        CONTEXT = max(CONTEXT, (DECODE_FROM + args.steps + max(3, args.warmup) + 64 + 63) // 64 * 64)      # whole pages

    if args.impl == "reference":
        # The reference is a C++/CMake program (pip: "neither setup.py nor pyproject.toml found"), so it was built
        # with its own CMake (-DEMBER_CUDA=ON -DCMAKE_CUDA_ARCHITECTURES=100: compiles and links) and driven through
        # create_backend("cuda") -> Backend::forward -> Backend::sample on this workload.  Its first step, a
        # 2,048-token prompt at these layer widths, ended with a memory fault on the B200, so its GPU code is not
        # run again here and this arm stays unavailable.
        print(json.dumps({"impl": "reference", "unavailable":
                          "the reference's CUDA backend, built unmodified with its own CMake for sm_100, faulted on a B200 "
                          "in its first step of this workload (2,048-token prompt, Qwen3-1.7B widths): 'CUDA error at "
                          "src/backend/cuda/cuda_backend.cu:214: an illegal memory access was encountered "
                          "(cudaStreamSynchronize(stream_))'; GPU code that faulted is not run again on this shared pool"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py measures one GPU (this engine is single-GPU); --gpus {args.gpus} is not supported")
        return 2
    warmup = max(3, args.warmup)

    import torch
    from ember_b200.config import Qwen3Config
    cfg = Qwen3Config.from_json(QWEN3_1P7B)
    n_layers = args.layers or cfg.num_hidden_layers
    pk = peaks()
    wbytes, kv_per_token, prefill_flops = model_bytes_and_flops(cfg, n_layers)

    if args.workload == "serving-8b":
        return workload_serving_8b(args, pk)
    if args.workload == "qwen3-32b":
        return workload_qwen3_32b(args, pk)
    if args.workload == "fadosun":
        return workload_fadosun(args, pk)
    if args.workload == "zufusun":
        return workload_zufusun(args, pk)
    if args.workload == "fomanex":
        return workload_fomanex(args, pk)
    if args.workload == "pepapel":
        return workload_pepapel(args, pk)
    if args.workload == "filanex":
        return workload_filanex(args, pk)
    if args.workload == "malusun":
        return workload_malusun(args, pk)
    if args.breakdown:
        return breakdown(cfg, n_layers, args.batch)
    if args.only_prefill:
        n_tok = max(2, args.prefill_tokens)
        llm = build_llm(cfg, n_layers, 1, prefill_tokens=n_tok)
        pms = time_prefill(llm, n_tok, reps=max(1, min(5, args.steps)), warmup=min(3, warmup))
        fl = prefill_flops(n_tok)
        print(json.dumps({"prefill": {"value": round(n_tok / (pms * 1e-3), 1), "tokens": n_tok,
                                      "ms": round(pms, 3), "tflops": round(fl / (pms * 1e-3) / 1e12, 1), "layers": n_layers}}))
        return 0

    room = CONTEXT - DECODE_FROM - 8                 # positions left for timed steps before the context limit
    with ClockSampler() as clocks_all:
        llm = build_llm(cfg, n_layers, max(args.batch, 1))
        with ClockSampler() as clocks:
            ms, launches, repeats, mean_ctx = time_decode(llm, args.batch, args.steps, warmup, DECODE_FROM, max_steps=min(900, room))
        # (the end-to-end loop prefills its prompts through the engine; at other context lengths than the default's
        # the first requests would be done decoding before the last has its prompt in, so it is measured at the
        # default only)
        e2e_ms, h2d, d2h = time_e2e(llm, args.batch, args.steps, warmup, DECODE_FROM) if custom_context is None else (None, 0, 0)
        value = args.batch * 1000.0 / ms
        step_bytes = wbytes + args.batch * mean_ctx * kv_per_token
        achieved = step_bytes / (ms * 1e-3) / 1e9
        head_clocks = clocks.summary()
        out = {
            "metric": "decode tok/s at batch 1/8/64; prefill tok/s at 2,048 tokens (Qwen3-1.7B)",
            "value": round(value, 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": warmup,
            "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
            "dtype": "bf16", "data": "synthetic (random weights from a seed, random token ids)", "impl": "ours",
            "config": {"model": "Qwen3-1.7B shape", "global_batch": args.batch, "seq_len": CONTEXT,
                       "decode_from": DECODE_FROM, "layers": n_layers, "layers_of_config": cfg.num_hidden_layers,
                       "hidden": cfg.hidden_size, "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads,
                       "head_dim": cfg.head_dim, "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size,
                       "tied": cfg.tie_word_embeddings, "page_tokens": PAGE_TOKENS, "parallelism": "single GPU",
                       "l2": "inputs larger than L2 (3.4 GB of weights per step); no flush",
                       "timing": f"median of {repeats} regions of {args.steps} steps, CUDA events",
                       "peaks": pk["source"]},
            "clocks": head_clocks,
            "e2e": ({"value": round(args.batch * 1000.0 / e2e_ms, 1), "unit": "tokens/s", "ms_per_step": round(e2e_ms, 4),
                     "h2d_bytes_per_step": int(h2d), "d2h_bytes_per_step": int(d2h)} if e2e_ms is not None else
                    {"skipped": "measured at the default context only"}),
            "gpu_launches": int(round(launches * args.steps)),
            "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                         "frac": round(achieved / pk["hbm_gbs"], 4), "bytes_per_step": int(step_bytes)},
        }
        if head_clocks.get("sm_mhz"):
            # time x clock: lets a run at boost clocks be compared with one under the power cap
            out["ms_per_step_x_ghz"] = round(ms * head_clocks["sm_mhz"] / 1000.0, 4)
        del llm
        torch.cuda.empty_cache()

        if not args.skip_points:
            llm = build_llm(cfg, n_layers, 1)
            pms = time_prefill(llm, PREFILL_TOKENS, reps=5, warmup=3)
            fl = prefill_flops(PREFILL_TOKENS)
            out["prefill"] = {"value": round(PREFILL_TOKENS / (pms * 1e-3), 1), "tokens": PREFILL_TOKENS, "ms": round(pms, 3),
                              "frac": round(fl / (pms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4), "tflops": round(fl / (pms * 1e-3) / 1e12, 1)}
            points, points_e2e, fracs = {}, {}, {}
            ms1, _, _, ctx1 = time_decode(llm, 1, args.steps, warmup, DECODE_FROM, max_steps=min(900, room))
            points["decode_b1"] = round(1000.0 / ms1, 1)
            fracs["decode_b1"] = round((wbytes + ctx1 * kv_per_token) / (ms1 * 1e-3) / 1e9 / pk["hbm_gbs"], 4)
            if custom_context is None:
                points_e2e["decode_b1"] = round(1000.0 / time_e2e(llm, 1, args.steps, warmup, DECODE_FROM)[0], 1)
            del llm
            torch.cuda.empty_cache()
            llm = build_llm(cfg, n_layers, 64)
            ms64, _, _, ctx64 = time_decode(llm, 64, max(8, args.steps // 2), warmup, DECODE_FROM, max_steps=min(900, room))
            points["decode_b64"] = round(64 * 1000.0 / ms64, 1)
            fracs["decode_b64"] = round((wbytes + 64 * ctx64 * kv_per_token) / (ms64 * 1e-3) / 1e9 / pk["hbm_gbs"], 4)
            if custom_context is None:
                points_e2e["decode_b64"] = round(64 * 1000.0 / time_e2e(llm, 64, max(8, args.steps // 2), warmup, DECODE_FROM)[0], 1)
            points["decode_b8"] = round(value, 1)
            fracs["decode_b8"] = out["roofline"]["frac"]
            if e2e_ms is not None:
                points_e2e["decode_b8"] = out["e2e"]["value"]
            out["points"] = points
            out["points_e2e"] = points_e2e
            out["points_hbm_frac"] = fracs
            del llm
    out["clocks_all_points"] = clocks_all.summary()
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
