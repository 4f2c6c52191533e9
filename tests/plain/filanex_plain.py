"""Plain, slow Filanex forward for whole sequences: no cache, no batching, no kernels.

One function per mechanism, written from the design's equations with torch on the CPU (float64 by default).  It shares
no code with ``ember_b200``: it takes the configuration as the dictionary config.json holds and the weights as a
name -> tensor dictionary.  Attention is a dense [T, T] score matrix under a boolean mask, the rotation works on the
pairs as they are stored, experts run one token at a time.

Notation: x [T, width] the residual stream, h a sublayer's input, W[name] a matrix stored [out, in].
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def lin(h: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = h @ w.to(h.dtype).T
    return y + b.to(h.dtype) if b is not None else y


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w.to(x.dtype)


# --------------------------------------------------------------------------------------------- embedding
def bigram_rows(tokens: List[int], bigram: dict) -> List[int]:
    """The hashed row of (token before, token) for every token; the first token has the row after the last bucket."""
    n, a, b = int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"])
    return [n if i == 0 else (tokens[i - 1] * a + t * b) % n for i, t in enumerate(tokens)]


def embed(config: dict, W: Dict[str, torch.Tensor], tokens: List[int], dtype) -> torch.Tensor:
    x = W["embed"].to(dtype)[torch.tensor(tokens, dtype=torch.long)]
    bigram = (config.get("embedding") or {}).get("bigram")
    if bigram:
        x = x + W["bigram"].to(dtype)[torch.tensor(bigram_rows(tokens, bigram), dtype=torch.long)]
    return x


# --------------------------------------------------------------------------------------------- positions
def frequencies(rot: dict, dtype):
    """(angle per position of every pair, factor of cosines and sines)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=dtype)
    f = base ** (-2.0 * i / dims)
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    factor, original = float(s["factor"]), float(s["original"])

    def dim_of(turns: float) -> float:
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(float(s["fast"]))), 0)
    hi = min(math.ceil(dim_of(float(s["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, dim]: elements 2i and 2i + 1 of the first rot.dims turn by p f_i; the rest passes."""
    dims = int(rot["dims"])
    f, mag = frequencies(rot, x.dtype)
    a = torch.arange(x.shape[0], dtype=x.dtype)[:, None] * f[None, :]
    c, s = (torch.cos(a) * mag)[:, None, :], (torch.sin(a) * mag)[:, None, :]
    y = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2] = u * c - v * s
    y[..., 1:dims:2] = v * c + u * s
    return y


def visible(T: int, chunk: int = 0) -> torch.Tensor:
    """[T, T] mask: j <= i, and with ``chunk`` both in the same chunk of positions."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    m = j <= i
    if chunk > 0:
        m = m & ((i // chunk) == (j // chunk))
    return m


# ------------------------------------------------------------------------------------------------- mixer
def capped_attention(q, k, v, scale: float, mask: torch.Tensor, softcap: float = 0.0) -> torch.Tensor:
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]; query head h reads key head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap > 0:
            s = softcap * torch.tanh(s / softcap)
        out.append(torch.softmax(s.masked_fill(~mask, float("-inf")), dim=-1) @ v[:, g])
    return torch.stack(out, dim=1)


def attention_mixer(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = lin(h, W[p + "q"]).reshape(T, H, D), lin(h, W[p + "k"]).reshape(T, G, D), lin(h, W[p + "v"]).reshape(T, G, V)
    if m.get("rot"):
        q, k = rotate_pairs(q, m["rot"]), rotate_pairs(k, m["rot"])
    mask = visible(T, int((m.get("mask") or {}).get("size", 0)))
    o = capped_attention(q, k, v, float(m["scale"]), mask, float(m.get("softcap") or 0.0)).reshape(T, H * V)
    return lin(o * torch.sigmoid(lin(h, W[p + "g"])), W[p + "o"])


# ----------------------------------------------------------------------------------------- feed-forwards
def gelu(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def dense_ff(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(gelu(lin(h, W[p + "up"], W[p + "up.b"])), W[p + "down"], W[p + "down.b"])


def route(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, router: dict):
    """(chosen [T, top], weights [T, top]): sigmoid scores; only the ``keep`` groups whose two largest scores have the
    largest sums can be chosen from; the chosen scores are divided by their sum."""
    top = int(router["top"])
    s = torch.sigmoid(lin(h, W[p + "router"]))
    c = s
    groups = router.get("groups")
    if groups:
        count, keep = int(groups["count"]), int(groups["keep"])
        per = s.shape[1] // count
        score = torch.topk(s.reshape(-1, count, per), min(2, per), dim=-1).values.sum(-1)
        kept = torch.zeros_like(score, dtype=torch.bool)
        kept.scatter_(1, torch.topk(score, keep, dim=-1).indices, True)
        c = s.masked_fill(~kept.repeat_interleave(per, dim=1), float("-inf"))
    chosen = torch.topk(c, top, dim=-1).indices
    w = torch.gather(s, 1, chosen)
    return chosen, w / (w.sum(-1, keepdim=True) + 1e-20)


def moe_ff(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, mlp: dict) -> torch.Tensor:
    chosen, weights = route(h, W, p, mlp["router"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weights[t]):
            z = lin(h[t:t + 1], W[f"{p}e{e}.gate"])
            y[t] += w * lin(z * torch.sigmoid(z) * lin(h[t:t + 1], W[f"{p}e{e}.up"]), W[f"{p}e{e}.down"])[0]
    return y


# ------------------------------------------------------------------------------------------------- model
def run_order(config: dict):
    """(layer, whether the stream is mixed with the embedding output before it) in the order they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    once = [(i, i == a) for i in range(a, b)]
    return [(i, False) for i in range(a)] + once * int(loop["times"]) + [(i, False) for i in range(b, n)]


def forward(config: dict, W: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64, layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) receives the stream after every layer run."""
    eps = float(config["norm"]["eps"])
    x = x0 = embed(config, W, tokens, dtype)
    for i, mix in run_order(config):
        if mix:
            x = lin(torch.cat([x, x0], dim=-1), W["loop.in"])
        layer, p = config["layers"][i], f"l{i}."
        if layer["type"] != "attention":
            raise ValueError(layer["type"])
        h = rms_norm(x, W[p + "norm1"], eps)
        y = attention_mixer(h, W, p + "mix.", layer["mixer"])
        mlp = layer.get("mlp")
        if mlp is not None:
            y = y + (dense_ff(h, W, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(h, W, p + "mlp.", mlp))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return lin(rms_norm(x, W["final.norm"], eps), W["head"])
