"""Malusun: a decoder whose layers are listed one by one in config.json, every sublayer between two norms: the
stream gains ``norm1b(mixer(norm1(.)))`` of itself and after it ``norm2b(ff(norm2(.)))``; norm weights are stored around zero.  Three mixers: a
selective scan with a diagonal state per channel ("mamba1"); grouped-query softmax attention in a sliding window with a
rotate-half rotation of part of each head ("attention"); and the same without a rotation, with biases, a linear distance
bias on the scores and one added to the softmax's denominator ("attention_2").  Attention layers may blend their values
with those of the first layer that does so.  Two feed-forwards: a dense one with relu squared, and a mixture of gated
experts with sigmoid scores that weigh an expert's *input*, beside a shared expert.  The embedding is multiplied by a
constant.

config.json keys: ``architecture`` "Malusun"; ``vocab``; ``width``; ``norm.eps``; ``embedding.scale`` (absent: 1); ``layers``: a
list of ``{"type", "mixer", "mlp"}`` where ``type`` is "mamba1" (mixer: inner, state, dt_rank, conv), "attention" (heads,
kv_heads, dim, vdim, scale, mask.size, rot {dims, base}, v_mix) or "attention_2" (the same without rot); mask, rot and
v_mix are optional; ``mlp`` is ``{"kind": "dense", "ff"}``, ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"},
"shared": {"ff"}}`` (shared optional) or null.  Tensor names: ``embed``, ``head``, ``final.norm`` and per layer ``l<i>.`` +
norm1, norm1b, norm2, norm2b, ``mix.in|conv|conv.b|x|dt|dt.b|A_log|D|o`` or ``mix.q|k|v`` (+ ``.b``), ``mix.vmix``, ``mix.o``,
``mlp.up|down`` or ``mlp.router``, ``mlp.e<j>.gate|up|down``, ``mlp.shared.gate|up|down``.

One optional key is this engine's own: ``max_positions`` (longest sequence; default 1,048,576).
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Mapping, Optional, Tuple

from .registry import register_architecture
from .spec import (ConfigError, LayerSpec, MLPSpec, ModelSpec, NoPositionSpec, PartSpec, RMSNormSpec, RotarySpec, RoutedMLPSpec,
                   SelectiveScanSpec, SinkAttentionSpec, default_schedule)
from .zufusun import _float, _int, _need

MIXERS = ("mamba1", "attention", "attention_2")
# fixed by the design: the exponents of the distance slopes run from 8 / heads to 8, and the sink's score is 0
SLOPE_SPAN = 8.0
SINK_SCORE = 0.0


@dataclass(frozen=True)
class MalusunConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: Tuple[dict, ...]            # as config.json lists them (checked)
    max_positions: int = 1 << 20

    architecture = "Malusun"
    model_type = "malusun"

    @classmethod
    def from_json(cls, config: Mapping, generation_config: Optional[Mapping] = None) -> "MalusunConfig":
        layers = _need(config, "layers", "the model")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        embedding = config.get("embedding") or {}
        out = cls(vocab=_int(config, "vocab", "the model"), width=_int(config, "width", "the model"),
                  eps=_float(_need(config, "norm", "the model"), "eps", "norm"),
                  embedding_scale=_float(embedding, "scale", "embedding") if embedding.get("scale") is not None else 1.0,
                  layers=tuple(copy.deepcopy(dict(l)) for l in layers),
                  max_positions=int(config.get("max_positions") or (1 << 20)))
        # every layer's keys are read and every part is built (without a device) now, so that a bad value is
        # refused here and not at the first step
        from ..model.causal_lm import CausalLM
        CausalLM(out.to_model_spec())
        return out

    # ------------------------------------------------------------------ parts
    def _norm(self) -> RMSNormSpec:
        return RMSNormSpec(size=self.width, eps=self.eps, weight_suffix="", weight_offset=1.0)

    def _kind(self, i: int) -> str:
        kind = _need(self.layers[i], "type", f"layers[{i}]")
        if kind not in MIXERS:
            raise ConfigError(f"config.json: layers[{i}].type {kind!r} is not a mixer of this design ({', '.join(MIXERS)})")
        return kind

    def mixes_values(self, i: int) -> bool:
        """Whether layer i takes part in the blending of values."""
        return self._kind(i) != "mamba1" and bool(_need(self.layers[i], "mixer", f"layers[{i}]").get("v_mix"))

    def value_source(self) -> int:
        """The first layer that takes part in it: the later ones blend with its values (-1: none does)."""
        return next((i for i in range(len(self.layers)) if self.mixes_values(i)), -1)

    def _mixer(self, i: int, m: Mapping) -> PartSpec:
        where, kind = f"layers[{i}].mixer", self._kind(i)
        if kind == "mamba1":
            return SelectiveScanSpec(hidden_size=self.width, inner=_int(m, "inner", where), state_size=_int(m, "state", where),
                                     dt_rank=_int(m, "dt_rank", where), conv_taps=_int(m, "conv", where))
        heads, dim, second = _int(m, "heads", where), _int(m, "dim", where), kind == "attention_2"
        kv, vdim = _int(m, "kv_heads", where), _int(m, "vdim", where)
        position, rot = NoPositionSpec(), m.get("rot")
        if not second and rot is not None and _int(rot, "dims", where + ".rot", least=0) > 0:
            position = RotarySpec(head_dim=dim, rotary_dim=_int(rot, "dims", where + ".rot"), theta=_float(rot, "base", where + ".rot"),
                                  frequency_precision="float64", layout="half")
        source, mix = self.value_source(), ""
        if self.mixes_values(i):
            mix = "source" if i == source else "mix"
            first = self.layers[source]["mixer"]
            if _int(first, "kv_heads", f"layers[{source}].mixer") * _int(first, "vdim", f"layers[{source}].mixer") != kv * vdim:
                raise ConfigError(f"config.json: {where}: values of {kv} x {vdim} cannot blend with those of layer {source}")
        mask = m.get("mask")
        return SinkAttentionSpec(
            hidden_size=self.width, num_heads=heads, num_kv_heads=kv, head_dim=dim, value_dim=vdim, scale=_float(m, "scale", where),
            bias=second, qk_norm="none", window=_int(mask, "size", where + ".mask") if mask is not None else 0, position=position,
            sink=second, fixed_sink=SINK_SCORE if second else None, slope_span=SLOPE_SPAN if second else 0.0, value_mix=mix)

    def _feed_forward(self, i: int, mlp: Mapping) -> PartSpec:
        where = f"layers[{i}].mlp"
        kind = mlp.get("kind")
        if kind == "dense":
            return MLPSpec(hidden_size=self.width, intermediate_size=_int(mlp, "ff", where), activation="square_relu",
                           names=("up", "down"))
        if kind == "moe":
            expert, router, shared = _need(mlp, "expert", where), _need(mlp, "router", where), mlp.get("shared")
            return RoutedMLPSpec(hidden_size=self.width, intermediate_size=_int(expert, "ff", where + ".expert"),
                                 experts=_int(router, "experts", where + ".router"), top=_int(router, "top", where + ".router"),
                                 limit=0.0, alpha=1.0, up_offset=0.0, scoring="sigmoid", weigh="input",
                                 shared_size=_int(shared, "ff", where + ".shared") if shared is not None else 0)
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not a feed-forward of this design (dense, moe)")

    # --------------------------------------------------------------- as a model
    def to_model_spec(self) -> ModelSpec:
        layers = []
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            parts = [("mixer_norm", self._norm(), p + "norm1"), ("mixer", self._mixer(i, _need(l, "mixer", f"layers[{i}]")), p + "mix."),
                     ("mixer_out_norm", self._norm(), p + "norm1b")]
            if l.get("mlp") is not None:
                parts += [("feed_forward_norm", self._norm(), p + "norm2"), ("feed_forward", self._feed_forward(i, l["mlp"]), p + "mlp."),
                          ("feed_forward_out_norm", self._norm(), p + "norm2b")]
            layers.append(LayerSpec("gated_sandwich", tuple(parts)))
        return ModelSpec(architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, layers=tuple(layers),
                         schedule=default_schedule(len(layers)), final_norm=self._norm(), final_norm_prefix="final.norm",
                         embedding_name="embed", head_name="head", tie_embeddings=False, head_optional=False,
                         max_positions=self.max_positions, eos_ids=(), init_std=0.05, init_norm_std=0.1,
                         embedding_multiplier=self.embedding_scale)

    def to_json(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "embedding": {"scale": self.embedding_scale}, "layers": [copy.deepcopy(l) for l in self.layers]}
        if self.max_positions != 1 << 20:
            d["max_positions"] = self.max_positions
        return d

    def _needs(self):
        from ..model.causal_lm import CausalLM
        return CausalLM(self.to_model_spec()).cache_needs()

    def kv_bytes_per_token(self, elem_bytes: int) -> int:
        """Bytes of paged cache one token takes (while inside the windows): keys and values of the attention layers."""
        return sum(n.num_kv_heads * (n.head_dim + (n.value_dim or n.head_dim)) * elem_bytes
                   for n in self._needs().values() if n is not None and n.kind in ("full", "window"))

    def state_bytes_per_request(self) -> int:
        """Bytes of fixed-size fp32 state one request holds: the scans' states and the convolutions' last inputs."""
        from ..cache.storage import state_bytes_per_request
        return state_bytes_per_request(self._needs())

    def describe(self) -> str:
        kinds = ", ".join(l["type"] for l in self.layers[:8]) + (", ..." if len(self.layers) > 8 else "")
        return f"malusun: {len(self.layers)} layers ({kinds}), width {self.width}, vocab {self.vocab}"


register_architecture(MalusunConfig.architecture, MalusunConfig, model_type=MalusunConfig.model_type)
