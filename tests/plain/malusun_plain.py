"""Plain, slow Malusun forward for whole sequences: no cache, no batching, no kernels.

One function per mechanism, written from the design's equations with torch on the CPU (float64 by default).  It shares
no code with ``ember_b200``: it takes the configuration as the dictionary config.json holds and the weights as a
name -> tensor dictionary.  Attention is a dense [T, T] score matrix under a boolean mask, the selective scan walks the
tokens one by one, experts run one token at a time.

Notation: x [T, width] the residual stream, h a sublayer's input, W[name] a matrix stored [out, in].
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


def lin(h: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = h @ w.to(h.dtype).T
    return y + b.to(h.dtype) if b is not None else y


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The stored weight is the distance from one."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * (1.0 + w.to(x.dtype))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


# ------------------------------------------------------------------------------------------ selective scan
def causal_conv(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, n]: y[t, c] = bias[c] + sum_j taps[c, j] x[t - (n - 1 - j), c], zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    padded = torch.cat([x.new_zeros(n - 1, x.shape[1]), x])
    y = bias.to(x.dtype).expand(T, -1).clone()
    for j in range(n):
        y = y + padded[j:j + T] * taps[:, j].to(x.dtype)
    return y


def selective_scan(x: torch.Tensor, dt: torch.Tensor, A: torch.Tensor, B: torch.Tensor, C: torch.Tensor, D: torch.Tensor,
                   S: Optional[torch.Tensor] = None):
    """x, dt [T, inner], A [inner, state], B, C [T, state], D [inner] -> (y [T, inner], last S [inner, state])."""
    S = torch.zeros_like(A) if S is None else S
    ys = []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        ys.append(S @ C[t] + D * x[t])
    return torch.stack(ys), S


def mamba_mixer(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict) -> torch.Tensor:
    inner, N, R = int(m["inner"]), int(m["state"]), int(m["dt_rank"])
    x, z = lin(h, W[p + "in"]).split([inner, inner], dim=-1)
    x = silu(causal_conv(x, W[p + "conv"], W[p + "conv.b"]))
    low, B, C = lin(x, W[p + "x"]).split([R, N, N], dim=-1)
    dt = torch.nn.functional.softplus(lin(low, W[p + "dt"], W[p + "dt.b"]), threshold=1e9)
    y, _ = selective_scan(x, dt, -torch.exp(W[p + "A_log"].to(h.dtype)), B, C, W[p + "D"].to(h.dtype))
    return lin(y * silu(z), W[p + "o"])


# ----------------------------------------------------------------------------------------------- attention
def rotate_half(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, dim]: elements i and i + dims / 2 of the first dims turn by p base^(-2i / dims); the rest passes."""
    dims, half = int(rot["dims"]), int(rot["dims"]) // 2
    f = float(rot["base"]) ** (-2.0 * torch.arange(half, dtype=x.dtype) / dims)
    a = (torch.arange(x.shape[0], dtype=x.dtype)[:, None] * f)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., dims:]], dim=-1)


def visible(T: int, window: int = 0) -> torch.Tensor:
    """[T, T] mask: 0 <= i - j, and i - j < window where there is one."""
    gap = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (gap >= 0) & ((gap < window) if window > 0 else True)


def slopes(heads: int) -> List[float]:
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def softmax_attention(q, k, v, scale: float, mask: torch.Tensor) -> torch.Tensor:
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]; query head h reads key head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~mask, float("-inf"))
        out.append(torch.softmax(s, dim=-1) @ v[:, g])
    return torch.stack(out, dim=1)


def biased_attention(q, k, v, scale: float, mask: torch.Tensor) -> torch.Tensor:
    """As above with slope_h * (i - j) taken off the scores and a one added to every denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    gap = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(q.dtype)
    out = []
    for h, slope in enumerate(slopes(H)):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale - slope * gap).masked_fill(~mask, float("-inf"))
        top = s.max(-1, keepdim=True).values.clamp(min=0.0)                 # (the sink's own score is 0)
        e = torch.exp(s - top)
        out.append((e @ v[:, g]) / (torch.exp(-top) + e.sum(-1, keepdim=True)))
    return torch.stack(out, dim=1)


def mix_values(v: torch.Tensor, first: torch.Tensor, lam: torch.Tensor) -> torch.Tensor:
    lam = lam.to(v.dtype)
    return (1.0 - lam) * v + lam * first


def attention_mixer(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, kind: str, m: dict, shared: dict) -> torch.Tensor:
    """``shared``: what layers hand to one another within a sequence (the first mixing layer's values)."""
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    second = kind == "attention_2"
    proj = lambda n, heads, size: lin(h, W[p + n], W[p + n + ".b"] if second else None).reshape(T, heads, size)     # noqa: E731
    q, k, v = proj("q", H, D), proj("k", G, D), proj("v", G, V)
    if m.get("v_mix"):
        if "values" in shared:
            v = mix_values(v, shared["values"], W[p + "vmix"])
        else:
            shared["values"] = v
    mask = visible(T, int((m.get("mask") or {}).get("size", 0)))
    if second:
        o = biased_attention(q, k, v, float(m["scale"]), mask)
    else:
        rot = m.get("rot")
        if rot and int(rot["dims"]) > 0:
            q, k = rotate_half(q, rot), rotate_half(k, rot)
        o = softmax_attention(q, k, v, float(m["scale"]), mask)
    return lin(o.reshape(T, H * V), W[p + "o"])


# ----------------------------------------------------------------------------------------- feed-forwards
def dense_ff(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(torch.relu(lin(h, W[p + "up"])) ** 2, W[p + "down"])


def expert(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(silu(lin(h, W[p + "gate"])) * lin(h, W[p + "up"]), W[p + "down"])


def route(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, top: int):
    """(chosen [T, top], weights [T, top]): the largest sigmoid scores, as they are."""
    s = torch.sigmoid(lin(h, W[p + "router"]))
    got = torch.topk(s, top, dim=-1)
    return got.indices, got.values


def moe_ff(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, mlp: dict) -> torch.Tensor:
    chosen, weights = route(h, W, p, int(mlp["router"]["top"]))
    y = expert(h, W, p + "shared.") if mlp.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weights[t]):
            y[t] += expert(w * h[t:t + 1], W, f"{p}e{e}.")[0]
    return y


# ------------------------------------------------------------------------------------------------- model
def forward(config: dict, W: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64, layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) receives the stream after every layer."""
    eps = float(config["norm"]["eps"])
    scale = float((config.get("embedding") or {}).get("scale", 1.0))
    x = W["embed"].to(dtype)[torch.tensor(tokens, dtype=torch.long)] * scale
    shared: dict = {}
    for i, layer in enumerate(config["layers"]):
        p, mlp = f"l{i}.", layer.get("mlp")
        h = rms_norm(x, W[p + "norm1"], eps)
        if layer["type"] == "mamba1":
            y = mamba_mixer(h, W, p + "mix.", layer["mixer"])
        elif layer["type"] in ("attention", "attention_2"):
            y = attention_mixer(h, W, p + "mix.", layer["type"], layer["mixer"], shared)
        else:
            raise ValueError(layer["type"])
        x = x + rms_norm(y, W[p + "norm1b"], eps)
        if mlp is not None:
            h = rms_norm(x, W[p + "norm2"], eps)
            y = dense_ff(h, W, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(h, W, p + "mlp.", mlp)
            x = x + rms_norm(y, W[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return lin(rms_norm(x, W["final.norm"], eps), W["head"])
