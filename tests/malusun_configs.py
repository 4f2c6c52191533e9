"""The tests' own small Malusun configurations.  They differ from one another in every size, in the order and number of
layers, in the constants, in which optional keys are there, and in which values happen to be equal (key and value sizes,
heads and key heads, experts and choices) or 1."""
from __future__ import annotations

import json
import os

import torch


def _mamba(inner, state, dt_rank, conv):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def _attention(heads, kv_heads, dim, vdim, scale, window=None, rot=None, v_mix=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    if v_mix is not None:
        m["v_mix"] = v_mix
    return m


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top, shared=None):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


MALUSUN = {
    # widths the tensor-core kernels take; the first layer that blends values is the second one, a layer in between keeps its
    # own; windows of 33 and 50 on pages of 16; a scan of sixteen states; 64-wide heads in the last layers (in bfloat16 they
    # run on the kernels Qwen3's attention uses)
    "a": dict(seed=20, json={
        "architecture": "Malusun", "vocab": 320, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 8.0},
        "layers": [
            _layer("mamba1", _mamba(256, 16, 8, 4), _moe(48, 6, 2, 64)),
            _layer("attention", _attention(4, 2, 32, 24, 0.2, 33, (16, 10000.0), True), _dense(96)),
            _layer("attention_2", _attention(6, 2, 16, 24, 0.3, 50, v_mix=True), _moe(32, 4, 1, 32)),
            _layer("attention", _attention(4, 2, 64, 64, 0.15, 40, (64, 500.0)), _moe(40, 5, 3)),
            _layer("attention_2", _attention(4, 1, 64, 64, 0.12, 70), _dense(64)),
        ]}),
    # a width no tensor-core product takes; odd sizes everywhere; a window of a page exactly and of two tokens; no
    # mask, no rotation; two taps and one (no carried input); no feed-forward in one layer; as many choices as experts
    "b": dict(seed=7, json={
        "architecture": "Malusun", "vocab": 257, "width": 100, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.5},
        "layers": [
            _layer("attention_2", _attention(3, 3, 40, 6, 0.16, None, v_mix=True), _dense(70)),
            _layer("mamba1", _mamba(77, 5, 3, 2), _moe(30, 3, 3, 20)),
            _layer("attention", _attention(6, 3, 12, 6, 0.3, 16, (2, 10000.0), True), None),
            _layer("attention_2", _attention(9, 3, 20, 6, 0.25, 2, v_mix=True), _moe(50, 5, 1, 10)),
            _layer("mamba1", _mamba(40, 1, 1, 1), _dense(33)),
        ]}),
    # head sizes of a real model's layers: 128-wide keys and values with eight query heads on one key head, a window longer
    # than the page, experts of 256; a scan of 24 states over 512 channels
    "c": dict(seed=11, json={
        "architecture": "Malusun", "vocab": 512, "width": 256, "norm": {"eps": 1e-6}, "embedding": {"scale": 16.0},
        "layers": [
            _layer("attention_2", _attention(8, 1, 128, 128, 0.0884, 100, v_mix=True), _moe(256, 8, 1, 256)),
            _layer("attention", _attention(6, 1, 128, 128, 0.09, 256, (64, 50000.0), True), _dense(512)),
            _layer("mamba1", _mamba(512, 24, 16, 4), _moe(128, 8, 2, 128)),
            _layer("attention_2", _attention(12, 4, 128, 64, 0.1, 300), _dense(384)),
        ]}),
    # scans of 40 and 140 states, with more taps than the rolling convolution takes; no embedding scale; blending switched
    # off by its key; a layer of one head
    "d": dict(seed=13, json={
        "architecture": "Malusun", "vocab": 99, "width": 64, "norm": {"eps": 1e-5},
        "layers": [
            _layer("mamba1", _mamba(72, 40, 24, 3), None),
            _layer("attention", _attention(8, 8, 8, 8, 0.35, 1, (8, 100.0), False), _moe(24, 4, 1)),
            _layer("mamba1", _mamba(33, 140, 5, 6), _dense(40)),
            _layer("attention_2", _attention(1, 1, 20, 36, 0.3, 17), _dense(20)),
        ]}),
}


def malusun_config(name: str):
    from ember_b200.config import MalusunConfig
    return MalusunConfig.from_json(MALUSUN[name]["json"])


def write_malusun_dir(name_or_json, out_dir: str, seed: int = 0, spread_router: float = 6.0) -> str:
    """A model folder with random weights.  The router matrices are scaled up so that a choice is seldom a close call, the
    queries so that the weights over keys are far from even; norms, biases and the steps' biases are not near their neutral
    values.  The first blending layer gets a factor that nothing should read."""
    from ember_b200.config import MalusunConfig
    from ember_b200.weights import write_model_dir
    from ember_b200.weights.safetensors_io import save_file
    from tests.plain.qwen3_plain import read_safetensors
    cfg_json = MALUSUN[name_or_json]["json"] if isinstance(name_or_json, str) else name_or_json
    seed = MALUSUN[name_or_json]["seed"] if isinstance(name_or_json, str) else seed
    cfg = MalusunConfig.from_json(cfg_json)
    write_model_dir(cfg, out_dir, seed=seed, dtype=torch.bfloat16)
    path = os.path.join(out_dir, "model.safetensors")
    W = read_safetensors(path)
    g = torch.Generator().manual_seed(seed + 1)
    for name in W:
        if name.endswith(".router"):
            W[name] = W[name].float() * spread_router
        elif name.endswith(".mix.q") or name.endswith(".mix.x"):
            W[name] = W[name].float() * 3.0
        elif ".norm" in name:
            W[name] = 0.2 * torch.randn(W[name].shape, generator=g)
        elif name.endswith((".q.b", ".k.b", ".v.b", ".conv.b")):
            W[name] = 0.4 * torch.randn(W[name].shape, generator=g)
        elif name.endswith(".dt.b"):
            W[name] = -3.0 + 1.5 * torch.randn(W[name].shape, generator=g)
    if cfg.value_source() >= 0:
        W[f"l{cfg.value_source()}.mix.vmix"] = torch.tensor(77.0)
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


def drawn_malusun(seed: int) -> dict:
    """A configuration drawn from a seed: 1 to 5 layers of any mixer with any feed-forward or none, sizes and constants from
    short lists that include ones no tensor-core kernel takes and values that are equal or 1."""
    import numpy as np
    rng = np.random.default_rng(seed)
    pick = lambda *v: v[int(rng.integers(0, len(v)))]                         # noqa: E731
    layers, (kv, vdim) = [], (pick(1, 2, 3), pick(16, 24, 32, 64, 128, 10))     # values that blend have one size
    for _ in range(int(rng.integers(1, 6))):
        k = rng.random()
        if k < 0.4:
            mlp = _dense(pick(64, 128, 200, 384, 50))
        elif k < 0.9:
            e = pick(1, 2, 4, 6, 8, 16, 33)
            mlp = _moe(pick(32, 64, 96, 40), e, int(rng.integers(1, min(e, 6) + 1)), pick(None, 32, 64, 50))
        else:
            mlp = None
        kind = pick("mamba1", "attention", "attention_2")
        if kind == "mamba1":
            mixer = _mamba(pick(64, 128, 320, 90, 51), pick(1, 4, 8, 16, 24, 33, 64), pick(1, 8, 12, 16, 32), pick(1, 2, 3, 4, 5, 9))
        else:
            mix = pick(True, True, False, None)
            dim = pick(16, 32, 64, 128, 24, 20, vdim)
            own_kv, own_v = (kv, vdim) if mix else (pick(1, 2, 3), pick(16, 48, 64, dim, dim))
            rot = (dim - dim % 2 if pick(True, False) else min(dim - dim % 2, pick(2, 8, 16)), pick(10000.0, 500.0, 1e6)) if kind == "attention" and rng.random() < 0.9 else None
            mixer = _attention(own_kv * pick(1, 2, 4), own_kv, dim, own_v, float(dim ** -0.5 * pick(1.0, 0.7, 2.0)),
                               pick(None, 16, 24, 50, 64, 96, 7, 1, 130), rot, mix)
        layers.append(_layer(kind, mixer, mlp))
    return {"architecture": "Malusun", "vocab": pick(384, 512, 640, 333), "width": pick(128, 256, 136, 200, 64, 90),
            "norm": {"eps": pick(1e-5, 1e-6)}, "embedding": {"scale": pick(1.0, 6.0, 11.3)}, "layers": layers}
