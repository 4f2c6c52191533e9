"""The tests' own small Filanex configurations.  They differ from one another in every size, in the order and number of
layers, in the constants, in which optional keys are there, and in which values happen to be equal (key and value sizes,
heads and key heads, experts and choices, groups and kept groups) or 1."""
from __future__ import annotations

import json
import os

import torch


def _rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def _attention(heads, kv_heads, dim, vdim, scale, softcap=None, chunk=None, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        m["softcap"] = softcap
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot is not None:
        m["rot"] = rot
    return m


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top, groups=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def _layer(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


FILANEX = {
    # widths the tensor-core kernels take; chunks of 40 (not a multiple of a page of 16), values wider than keys, a partial
    # rotation; a loop in the middle of which the second layer has no feed-forward; 64-wide heads in the last layer (in
    # bfloat16 they run on the kernels Qwen3's attention uses); three groups of which two stay
    "a": dict(seed=3, json={
        "architecture": "Filanex", "vocab": 320, "width": 128, "norm": {"eps": 1e-6},
        "embedding": {"bigram": {"buckets": 211, "mul_prev": 7, "mul_cur": 3}}, "loop": {"start": 1, "stop": 3, "times": 2},
        "layers": [
            _layer(_attention(4, 2, 32, 48, 0.2, 20.0, 40, _rot(16, 10000.0, (4.0, 64, 16.0, 1.0))), _moe(48, 6, 2, (3, 2))),
            _layer(_attention(4, 1, 32, 16, 0.18, 6.0, 33, _rot(32, 500.0, (8.0, 100, 4.0, 2.0))), _dense(96)),
            _layer(_attention(2, 2, 16, 16, 0.25, 40.0, 24, _rot(8, 1000.0)), None),
            _layer(_attention(4, 2, 64, 64, 0.15, 10.0, 50, _rot(32, 10000.0, (2.0, 32, 8.0, 0.5))), _moe(32, 4, 3, (2, 2))),
        ]}),
    # a width no tensor-core product takes; odd head sizes; one head; a chunk of a page exactly and chunks of three
    # tokens; a loop over every layer; as many choices as experts, a single choice, groups of one; caps that bind; a
    # hash whose buckets are few and whose multipliers exceed them; no cap, no mask or no rotation in some layers
    "b": dict(seed=7, json={
        "architecture": "Filanex", "vocab": 257, "width": 100, "norm": {"eps": 1e-5},
        "embedding": {"bigram": {"buckets": 13, "mul_prev": 1000003, "mul_cur": 999983}}, "loop": {"start": 0, "stop": 4, "times": 3},
        "layers": [
            _layer(_attention(1, 1, 40, 24, 0.16, 2.0, 16, _rot(40, 77.0, (16.0, 512, 32.0, 1.0))), _dense(70)),
            _layer(_attention(6, 3, 12, 20, 0.3, None, 70, _rot(2, 10000.0)), _moe(30, 5, 1, (5, 1))),
            _layer(_attention(3, 3, 24, 8, 0.2, 5.0, 3), _moe(50, 3, 3)),
            _layer(_attention(5, 1, 20, 28, 0.22, 1.0, None, _rot(20, 1e6, (1.0, 16, 2.0, 1.0))), _moe(20, 8, 2, (4, 3))),
        ]}),
    # head sizes of a real model's layers: 128-wide keys and values, eight query heads on one key head, chunks of 256,
    # experts of 256; no bigram embedding; a loop over the last layer alone, run once
    "c": dict(seed=11, json={
        "architecture": "Filanex", "vocab": 512, "width": 256, "norm": {"eps": 1e-6}, "loop": {"start": 2, "stop": 3, "times": 1},
        "layers": [
            _layer(_attention(8, 1, 128, 128, 0.0884, 25.0, 256, _rot(64, 10000.0, (4.0, 256, 32.0, 1.0))), _moe(256, 8, 2, (4, 2))),
            _layer(_attention(6, 2, 128, 128, 0.09, 50.0, 100, _rot(128, 50000.0, (8.0, 1024, 32.0, 1.0))), _dense(512)),
            _layer(_attention(2, 1, 64, 128, 0.125, 30.0, 77, _rot(16, 10000.0)), _dense(384)),
        ]}),
    # every layer once: no loop, and the embedding's key is there without a bigram
    "d": dict(seed=13, json={
        "architecture": "Filanex", "vocab": 99, "width": 64, "norm": {"eps": 1e-5}, "embedding": {},
        "layers": [
            _layer(_attention(2, 1, 32, 32, 0.18, 8.0, 20, _rot(30, 100.0, (3.0, 20, 2.0, 1.0))), _dense(40)),
            _layer(_attention(8, 8, 8, 8, 0.35, 12.0, 1, _rot(8, 100.0)), _moe(24, 4, 1, (1, 1))),
        ]}),
}


def filanex_config(name: str):
    from ember_b200.config import FilanexConfig
    return FilanexConfig.from_json(FILANEX[name]["json"])


def write_filanex_dir(name_or_json, out_dir: str, seed: int = 0, spread_router: float = 6.0) -> str:
    """A model folder with random weights.  The router matrices are scaled up so that a choice is seldom a close call, the
    bigram rows are as large as the embedding's, the gates' matrices large enough to open and close, and the biases are
    not zero."""
    from ember_b200.config import FilanexConfig
    from ember_b200.weights import write_model_dir
    from ember_b200.weights.safetensors_io import save_file
    from tests.plain.qwen3_plain import read_safetensors
    cfg_json = FILANEX[name_or_json]["json"] if isinstance(name_or_json, str) else name_or_json
    seed = FILANEX[name_or_json]["seed"] if isinstance(name_or_json, str) else seed
    write_model_dir(FilanexConfig.from_json(cfg_json), out_dir, seed=seed, dtype=torch.bfloat16)
    path = os.path.join(out_dir, "model.safetensors")
    W = read_safetensors(path)
    g = torch.Generator().manual_seed(seed + 1)
    for name in W:
        if name.endswith(".router"):
            W[name] = (W[name].float() * spread_router).bfloat16()
        if name.endswith(".mix.g"):
            W[name] = (W[name].float() * 3.0).bfloat16()
        if name.endswith(".b") and W[name].dim() == 1:
            W[name] = (0.2 * torch.randn(W[name].shape, generator=g)).bfloat16()
        if name == "loop.in":                                # near [0.7, 0.5] x the identity: a pass keeps the stream's size
            n = W[name].shape[0]
            W[name] = (0.5 * W[name].float() + torch.cat([0.7 * torch.eye(n), 0.5 * torch.eye(n)], dim=1)).bfloat16()
    save_file({k: (v.bfloat16() if v.is_floating_point() else v) for k, v in W.items()}, path)
    with open(os.path.join(out_dir, "config.json"), "w") as f:        # the keys exactly as the test wrote them
        json.dump(cfg_json, f)
    return out_dir


def plain_inputs(model_dir: str):
    """(config dictionary, name -> float64 tensor) as the plain implementation takes them."""
    from tests.plain.qwen3_plain import read_safetensors
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    W = read_safetensors(os.path.join(model_dir, "model.safetensors"))
    return cfg, {k: (v.double() if v.is_floating_point() else v) for k, v in W.items()}


def drawn_filanex(seed: int) -> dict:
    """A configuration drawn from a seed: 1 to 5 layers with any feed-forward or none, any loop or none, with or without a
    bigram, sizes and constants from short lists that include ones no tensor-core kernel takes and values that are equal
    or 1."""
    import numpy as np
    rng = np.random.default_rng(seed)
    pick = lambda *v: v[int(rng.integers(0, len(v)))]                         # noqa: E731
    n, layers = int(rng.integers(1, 6)), []
    for _ in range(n):
        k = rng.random()
        if k < 0.4:
            mlp = _dense(pick(64, 128, 200, 384, 50))
        elif k < 0.9:
            e = pick(1, 2, 4, 6, 8, 16, 33)
            counts = [c for c in (1, 2, 3, 4, 8, 11) if e % c == 0]
            groups = None
            if rng.random() < 0.7:
                c = counts[int(rng.integers(0, len(counts)))]
                groups = (c, int(rng.integers(1, c + 1)))
            most = e if groups is None else groups[1] * (e // groups[0])
            mlp = _moe(pick(32, 64, 96, 40), e, int(rng.integers(1, min(most, 6) + 1)), groups)
        else:
            mlp = None
        kv, dim = pick(1, 2, 3), pick(16, 32, 64, 128, 24, 20)
        dims = pick(dim, dim // 2, 8, 4, 2)
        scaling = None if rng.random() < 0.3 else (pick(1.0, 2.0, 4.0, 16.0), pick(16, 100, 512, 4096), pick(32.0, 8.0, 2.0), pick(1.0, 0.5, 2.0))
        rot = None if rng.random() < 0.1 else _rot(dims - dims % 2, pick(10000.0, 500.0, 1e6, 20.0), scaling)
        layers.append(_layer(_attention(kv * pick(1, 2, 4), kv, dim, pick(16, 32, 48, 64, dim, dim), float(dim ** -0.5 * pick(1.0, 0.7, 2.0)),
                                        pick(None, 3.0, 30.0, 50.0), pick(None, 16, 24, 50, 64, 96, 7, 1, 130), rot), mlp))
    c = {"architecture": "Filanex", "vocab": pick(384, 512, 640, 333), "width": pick(128, 192, 256, 136, 200, 64, 90), "norm": {"eps": pick(1e-5, 1e-6)},
         "layers": layers}
    if rng.random() < 0.8:
        c["embedding"] = {"bigram": {"buckets": pick(1, 50, 509, 4096), "mul_prev": pick(1, 31, 7919), "mul_cur": pick(1, 17, 104729)}}
    if rng.random() < 0.7:
        a = int(rng.integers(0, n))
        c["loop"] = {"start": a, "stop": int(rng.integers(a + 1, n + 1)), "times": pick(1, 2, 3)}
    return c
