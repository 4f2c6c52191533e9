"""Filanex: a decoder whose layers are listed one by one in config.json, each with a single norm whose output both
sublayers read: ``h = norm1(x); x = x + (mixer(h) + ff(h))``.  The mixer is grouped-query softmax attention inside chunks
of positions: rotary positions in neighbouring pairs with frequencies stretched for long contexts, scores capped by a
tanh, and a sigmoid gate on every element of the concatenated heads.  Two feed-forwards: a dense one of two matrices
with biases and the exact gelu, and a mixture of gated experts with sigmoid scores, a limit to the groups of neighbouring
experts whose two best scores sum highest, and weights divided by their sum.  The embedded token gets a hashed embedding
of (previous token, token) added.  A stretch of layers may run several times in a row with the same weights and a cache of
its own for every pass; before each pass the stream is mixed with the embedding's output by a linear map of both.  The
logits are ``head`` applied to the RMS-normed stream.

config.json keys: ``architecture`` "Filanex"; ``vocab``; ``width``; ``norm.eps``; ``embedding.bigram`` {buckets, mul_prev,
mul_cur} (absent: none); ``loop`` {start, stop, times} (absent: every layer once, and no re-entry); ``layers``: a list of
``{"type", "mixer", "mlp"}`` where ``type`` is "attention" (mixer: heads, kv_heads, dim, vdim, scale, softcap, mask.size, rot
{dims, base, scaling {factor, original, fast, slow}}; softcap, mask, rot and its scaling are optional), and ``mlp`` is
``{"kind": "dense", "ff"}``, ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "groups": {"count", "keep"}}}`` or
null.  Tensor names: ``embed``, ``bigram``, ``loop.in``, ``head``, ``final.norm`` and per layer ``l<i>.`` + norm1,
``mix.q|k|v|g|o``, ``mlp.up|down`` (+ ``.b``) or ``mlp.router``, ``mlp.e<j>.gate|up|down``.

One optional key is this engine's own: ``max_positions`` (longest sequence; default 1,048,576).
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Mapping, Optional, Tuple

from .registry import register_architecture
from .spec import (BigramEmbeddingSpec, ConcatReentrySpec, ConfigError, LayerSpec, MLPSpec, ModelSpec, NoPositionSpec,
                   RMSNormSpec, RotarySpec, RoutedMLPSpec, ScheduleEntry, SinkAttentionSpec)
from .zufusun import _float, _int, _need

MIXERS = ("attention",)
RENORM_EPS = 1e-20           # added to the sum of the chosen experts' scores: fixed by the design


@dataclass(frozen=True)
class FilanexConfig:
    vocab: int
    width: int
    eps: float
    bigram: Optional[Tuple[int, int, int]]        # (buckets, mul_prev, mul_cur) or None
    loop: Optional[Tuple[int, int, int]]          # (start, stop, times) or None
    layers: Tuple[dict, ...]            # as config.json lists them (checked)
    max_positions: int = 1 << 20

    architecture = "Filanex"
    model_type = "filanex"

    @classmethod
    def from_json(cls, config: Mapping, generation_config: Optional[Mapping] = None) -> "FilanexConfig":
        layers = _need(config, "layers", "the model")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        loop = None
        if config.get("loop") is not None:
            lp = config["loop"]
            loop = (_int(lp, "start", "loop", least=0), _int(lp, "stop", "loop", least=0), _int(lp, "times", "loop", least=1))
            if not loop[0] < loop[1] <= len(layers):
                raise ConfigError(f"config.json: loop {loop[0]}..{loop[1]} is no stretch of the {len(layers)} layers")
        bigram = (config.get("embedding") or {}).get("bigram")
        if bigram is not None:
            w = "embedding.bigram"
            bigram = (_int(bigram, "buckets", w), _int(bigram, "mul_prev", w, least=0), _int(bigram, "mul_cur", w, least=0))
        out = cls(vocab=_int(config, "vocab", "the model"), width=_int(config, "width", "the model"),
                  eps=_float(_need(config, "norm", "the model"), "eps", "norm"), bigram=bigram, loop=loop,
                  layers=tuple(copy.deepcopy(dict(l)) for l in layers),
                  max_positions=int(config.get("max_positions") or (1 << 20)))
        # every layer's keys are read and every part is built (without a device) now, so that a bad value is
        # refused here and not at the first step
        from ..model.causal_lm import CausalLM
        CausalLM(out.to_model_spec())
        return out

    # ------------------------------------------------------------------ parts
    def _norm(self) -> RMSNormSpec:
        return RMSNormSpec(size=self.width, eps=self.eps, weight_suffix="")

    def _mixer(self, i: int, kind: str, m: Mapping) -> SinkAttentionSpec:
        where = f"layers[{i}].mixer"
        if kind not in MIXERS:
            raise ConfigError(f"config.json: layers[{i}].type {kind!r} is not a mixer of this design ({', '.join(MIXERS)})")
        dim = _int(m, "dim", where)
        position, rot = NoPositionSpec(), m.get("rot")
        if rot is not None and _int(rot, "dims", where + ".rot", least=0) > 0:
            scaling, sc = {}, rot.get("scaling")
            if sc is not None:
                w = where + ".rot.scaling"
                scaling = dict(scaling_factor=_float(sc, "factor", w), scaling_original=_float(sc, "original", w),
                               scaling_fast=_float(sc, "fast", w), scaling_slow=_float(sc, "slow", w))
            position = RotarySpec(head_dim=dim, rotary_dim=_int(rot, "dims", where + ".rot"), theta=_float(rot, "base", where + ".rot"),
                                  frequency_precision="float64", layout="interleaved", **scaling)
        mask = m.get("mask")
        return SinkAttentionSpec(
            hidden_size=self.width, num_heads=_int(m, "heads", where), num_kv_heads=_int(m, "kv_heads", where), head_dim=dim,
            value_dim=_int(m, "vdim", where), scale=_float(m, "scale", where), bias=False, qk_norm="none", sink=False,
            position=position, softcap=_float(m, "softcap", where) if m.get("softcap") is not None else 0.0,
            chunk=_int(mask, "size", where + ".mask") if mask is not None else 0, element_gate=True)

    def _feed_forward(self, i: int, mlp: Mapping):
        where = f"layers[{i}].mlp"
        kind = mlp.get("kind")
        if kind == "dense":
            return MLPSpec(hidden_size=self.width, intermediate_size=_int(mlp, "ff", where), activation="gelu",
                           names=("up", "down"), bias=True, bias_suffix=".b")
        if kind == "moe":
            expert, router = _need(mlp, "expert", where), _need(mlp, "router", where)
            groups, g = router.get("groups"), where + ".router.groups"
            return RoutedMLPSpec(hidden_size=self.width, intermediate_size=_int(expert, "ff", where + ".expert"),
                                 experts=_int(router, "experts", where + ".router"), top=_int(router, "top", where + ".router"),
                                 limit=0.0, alpha=1.0, up_offset=0.0, scoring="sigmoid", correction=False, route_scale=1.0,
                                 renormalize=True, renorm_eps=RENORM_EPS,
                                 groups=_int(groups, "count", g) if groups is not None else 0,
                                 keep_groups=_int(groups, "keep", g) if groups is not None else 0, group_score="top2")
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not a feed-forward of this design (dense, moe)")

    def order(self) -> Tuple[Tuple[int, int, bool], ...]:
        """(layer, pass, whether the stream re-enters before it) in run order."""
        n = len(self.layers)
        if self.loop is None:
            return tuple((i, 0, False) for i in range(n))
        a, b, times = self.loop
        return (tuple((i, 0, False) for i in range(a)) + tuple((i, t, i == a) for t in range(times) for i in range(a, b))
                + tuple((i, 0, False) for i in range(b, n)))

    # --------------------------------------------------------------- as a model
    def to_model_spec(self) -> ModelSpec:
        layers = []
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            kind, m = _need(l, "type", f"layers[{i}]"), _need(l, "mixer", f"layers[{i}]")
            parts = [("norm", self._norm(), p + "norm1"), ("mixer", self._mixer(i, kind, m), p + "mix.")]
            if l.get("mlp") is not None:
                parts.append(("feed_forward", self._feed_forward(i, l["mlp"]), p + "mlp."))
            layers.append(LayerSpec("parallel_prenorm", tuple(parts)))
        schedule = tuple(ScheduleEntry(i, instance=t, reentry=r) for i, t, r in self.order())
        return ModelSpec(architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, layers=tuple(layers),
                         schedule=schedule, final_norm=self._norm(), final_norm_prefix="final.norm",
                         embedding_name="embed", head_name="head", tie_embeddings=False, head_optional=False,
                         max_positions=self.max_positions, eos_ids=(), init_std=0.05, init_norm_std=0.1,
                         embedding_term=BigramEmbeddingSpec(size=self.width, buckets=self.bigram[0], mul_prev=self.bigram[1],
                                                            mul_cur=self.bigram[2]) if self.bigram is not None else None,
                         reentry=ConcatReentrySpec(size=self.width, name="loop.in") if self.loop is not None else None)

    def to_json(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "layers": [copy.deepcopy(l) for l in self.layers]}
        if self.bigram is not None:
            d["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        if self.max_positions != 1 << 20:
            d["max_positions"] = self.max_positions
        return d

    def _needs(self):
        from ..model.causal_lm import CausalLM
        return CausalLM(self.to_model_spec()).cache_needs()

    def kv_bytes_per_token(self, elem_bytes: int) -> int:
        """Bytes of paged cache one token takes: keys and values of every run of every layer."""
        return sum(n.num_kv_heads * (n.head_dim + (0 if n.keys_only else (n.value_dim or n.head_dim))) * elem_bytes
                   for n in self._needs().values() if n is not None and n.kind in ("full", "window"))

    def state_bytes_per_request(self) -> int:
        """Bytes of fixed-size state one request holds: its previous token."""
        from ..cache.storage import state_bytes_per_request
        return state_bytes_per_request(self._needs())

    def describe(self) -> str:
        loop = f", layers {self.loop[0]}..{self.loop[1] - 1} x {self.loop[2]}" if self.loop else ""
        return f"filanex: {len(self.layers)} layers{loop}, width {self.width}, vocab {self.vocab}"


register_architecture(FilanexConfig.architecture, FilanexConfig, model_type=FilanexConfig.model_type)
