"""What is added to the embedded tokens, and how the stream re-enters a looped stretch of layers.

* "bigram" (family "embedding_term"): a hashed embedding of (previous token, token), out = scale table[token] +
  bigram[(mul_prev previous + mul_cur token) mod buckets]; the first token of a sequence takes the table's last row.  One
  kernel gathers and adds both rows.  The previous token of a run's first token lies in the request's state slot (one
  int32), where the run's last token is left for the next step; the kernel reads tokens and slots on the device, so a
  decode step that is captured into a graph, or launched before its token has come back to the host, finds them too.
* "concat_linear" (family "reentry"): x <- W [x; x0] with x0 the embedding's output, ahead of every pass of a loop.  Both
  halves lie side by side in one operand row, so the map is a single product; x0's half is written once a step.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import ops
from ..config.spec import ConfigError
from .base import CacheNeed, EmbeddingTerm, Reentry, Runtime, WeightDecl
from .linear import Linear
from .registry import register_part


class BigramEmbedding(EmbeddingTerm):
    graph_safe = True

    def __init__(self, spec, prefix: str = ""):
        super().__init__(spec, prefix)
        s = spec
        if s.size <= 0 or s.buckets <= 0 or s.mul_prev < 0 or s.mul_cur < 0 or max(s.buckets, s.mul_prev, s.mul_cur) >= 1 << 31:
            raise ConfigError(f"bigram embedding: {s.buckets} buckets, multipliers {s.mul_prev} and {s.mul_cur} (each below 2^31)")

    def weight_decls(self) -> List[WeightDecl]:
        return [WeightDecl(self.prefix + self.spec.name, (self.spec.buckets + 1, self.spec.size))]

    def load(self, store, rt: Runtime) -> None:
        t = store.take(self.prefix + self.spec.name, (self.spec.buckets + 1, self.spec.size))
        if t is not None:
            self.table = rt.to_device(t, rt.weight_dtype(t.dtype))

    def cache_needs(self) -> Dict[str, Optional[CacheNeed]]:
        return {"bigram": CacheNeed(kind="state", state_shape=(1,), state_dtype="int32")}

    def embed(self, ctx, table: torch.Tensor, scale: float, out: torch.Tensor, caches) -> None:
        s = self.spec
        ops.embed_bigram(ctx.tokens, table, self.table, out, s.buckets, s.mul_prev, s.mul_cur, ctx.positions, ctx.seq_of,
                         ctx.query_start, ctx.state_slots, caches["bigram"].state, scale=scale, err=ctx.err, stream=ctx.stream,
                         prev_ids=ctx.prev_ids)


class ConcatReentry(Reentry):
    graph_safe = True

    def weight_decls(self) -> List[WeightDecl]:
        return [WeightDecl(self.prefix + self.spec.name, (self.spec.size, 2 * self.spec.size))]

    def load(self, store, rt: Runtime) -> None:
        self.rt = rt
        t = store.take(self.prefix + self.spec.name, (self.spec.size, 2 * self.spec.size))
        if t is not None:
            self.linear = Linear.from_host(t, rt)

    def _rows(self, ctx) -> torch.Tensor:
        return ctx.buf("reentry.rows", (ctx.max_tokens, 2 * self.spec.size), self.rt.dtype)       # [x | x0]

    def keep(self, ctx, h: torch.Tensor) -> None:
        ops.place_columns(h, self._rows(ctx), ctx.T, self.spec.size, stream=ctx.stream)

    def forward(self, ctx, h: torch.Tensor, first: bool = False) -> None:
        rows = self._rows(ctx)
        ops.place_columns(h, rows, ctx.T, 0, self.spec.size if first else -1, stream=ctx.stream)
        self.linear(ctx, rows, h, ctx.T, ops.EPI_STORE_F32)


register_part("embedding_term", "bigram", BigramEmbedding)
register_part("reentry", "concat_linear", ConcatReentry)
