"""Token embedding and output head.

Embedding: ``residual[t, :] = float32(E[id_t, :])``, no scale (reference:
runtime/backends/cuda/native/cuda_kernels.cu:599-614).  Output head:
``logits = x W^T`` with ``W = lm_head.weight [V, H]`` or the embedding table
when the head is tied (reference falls back to the embedding when
``lm_head.weight`` is absent, runtime/backends/cuda/native/weight_map.cpp:33-37);
logits come out in float32 (the reference rounds them to 16 bits first,
transformer_forward.cu:2178-2189).
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..config.registry import register_part
from ..kernels import ops
from ..weights.loader import IGNORED, MATRIX, VECTOR, WeightSpec
from .base import Part, StateNeed
from .linear import Linear
from .state_space import describe_row_entries


class TokenEmbedding(Part):
    """params: ``vocab``, ``hidden``, ``name`` (weight ``<name>.weight``) or ``weight_name`` (the table's full name),
    ``scale`` (default 1: the float32 row is multiplied by it)."""

    family = "embedding"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.vocab, self.hidden = int(params["vocab"]), int(params["hidden"])
        self.scale = float(params.get("scale", 1.0))
        self.table: torch.Tensor = None

    @classmethod
    def _table_name(cls, prefix, params) -> str:
        return params.get("weight_name") or cls.full_name(prefix, params, "weight")

    @classmethod
    def weight_specs(cls, params, prefix) -> List[WeightSpec]:
        return [WeightSpec(cls._table_name(prefix, params), (int(params["vocab"]), int(params["hidden"])), MATRIX,
                           std=float(params.get("std", 0.02)))]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.table = tensors[self._table_name(self.prefix, self.params)].contiguous()

    def forward(self, token_ids: torch.Tensor) -> torch.Tensor:
        out = torch.empty((token_ids.numel(), self.hidden), dtype=torch.float32, device=token_ids.device)
        return ops.embed_gather(self.table, token_ids, out, self.scale)

    def forward_step(self, ctx) -> torch.Tensor:
        return self.forward(ctx.token_ids)


class SinusoidNormEmbedding(Part):
    """Token embedding plus a sinusoidal position vector, then a layer norm:

        x = E[id] + P(pos),  P[2i] = sin(pos * base^(-2i/hidden)),  P[2i+1] = cos(the same angle)
        out = (x - mean) / sqrt(var + eps) * w

    in one kernel (angles in float64, the rest float32).  params: ``vocab``,
    ``hidden``, ``eps``, ``base`` (default 10000), ``table`` and
    ``norm_weight`` (the full names of the two tensors)."""

    family = "embedding"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.vocab, self.hidden = int(params["vocab"]), int(params["hidden"])
        self.eps, self.base = float(params["eps"]), float(params.get("base", 10000.0))
        self.table: torch.Tensor = None
        self.weight: torch.Tensor = None

    @classmethod
    def weight_specs(cls, params, prefix) -> List[WeightSpec]:
        v, h = int(params["vocab"]), int(params["hidden"])
        return [WeightSpec(params["table"], (v, h), MATRIX, std=float(params.get("std", 0.02))),
                WeightSpec(params["norm_weight"], (h,), VECTOR, init="one_plus_normal")]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.table = tensors[self.params["table"]].contiguous()
        self.weight = tensors[self.params["norm_weight"]].to(torch.float32).contiguous()

    def forward_step(self, ctx) -> torch.Tensor:
        out = torch.empty((ctx.token_ids.numel(), self.hidden), dtype=torch.float32, device=ctx.token_ids.device)
        return ops.embed_sinusoid_layernorm(self.table, ctx.token_ids, ctx.positions, self.weight, self.eps, self.base, out)


class BigramEmbedding(Part):
    """Token embedding plus, with ``bigram``, a hashed embedding of the token pair, for a stream of several copies:

        x = E[id] + B[(previous * mul_prev + id * mul_cur) mod buckets]      B[buckets] for a sequence's first token

    written to every copy of the stream.  Ids and the hash are 64-bit integers, the sum float32.  The last token of a
    portion waits in the request's state slot (stored one up, so that a zeroed slot says that there is none yet).
    params: ``vocab``, ``hidden``, ``table`` and ``pairs`` (the full names of the two tensors), ``bigram`` (None, or
    {buckets, mul_prev, mul_cur}), ``streams`` (default 1).  State: ``last_token`` int32 ``[1]``."""

    family = "embedding"
    describe_key = "row_entries"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.vocab, self.hidden, self.streams = int(params["vocab"]), int(params["hidden"]), int(params.get("streams") or 1)
        b = params.get("bigram")
        self.hash = (int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])) if b else None
        self.table: torch.Tensor = None
        self.pairs: torch.Tensor = None
        self.states: Dict[str, torch.Tensor] = {}

    @classmethod
    def weight_specs(cls, params, prefix) -> List[WeightSpec]:
        h = int(params["hidden"])
        specs = [WeightSpec(params["table"], (int(params["vocab"]), h), MATRIX)]
        if params.get("bigram"):
            specs.append(WeightSpec(params["pairs"], (int(params["bigram"]["buckets"]) + 1, h), MATRIX))
        return specs

    @classmethod
    def state_needs(cls, params) -> List[StateNeed]:
        return [StateNeed("last_token", (1,), torch.int32)] if params.get("bigram") else []

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.table = tensors[self.params["table"]].contiguous()
        if self.hash:
            self.pairs = tensors.pop(self.params["pairs"]).to(self.table.dtype).contiguous()

    def describe_step(self, layout, put) -> torch.Tensor:
        return describe_row_entries(layout, put)

    def forward_step(self, ctx) -> torch.Tensor:
        out = torch.empty((ctx.token_ids.numel(), self.streams, self.hidden), dtype=torch.float32, device=ctx.token_ids.device)
        return ops.embed_bigram(self.table, self.pairs, self.hash, ctx.token_ids, self.states.get("last_token"),
                                ctx.extras[self.describe_key], ctx.entry_q_start, ctx.entry_q_len, ctx.entry_slot, out)


class LinearHead(Part):
    """params: ``vocab``, ``hidden``, ``name``, ``tied_to`` (None, or the full
    name of the embedding table to use instead of a weight of its own),
    ``weight_name`` (the weight's full name where it is not ``<name>.weight``),
    ``scale`` (a factor on the float32 logits, default 1), ``softcap`` (None, or c: the logits become
    ``c * tanh(logits / c)``)."""

    family = "lm_head"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.vocab, self.hidden = int(params["vocab"]), int(params["hidden"])
        self.scale = float(params.get("scale", 1.0) or 1.0)
        self.softcap = float(params.get("softcap") or 0.0)
        self.linear: Linear = None

    @classmethod
    def _own_name(cls, prefix, params) -> str:
        return params.get("weight_name") or cls.full_name(prefix, params, "weight")

    @classmethod
    def weight_specs(cls, params, prefix) -> List[WeightSpec]:
        shape = (int(params["vocab"]), int(params["hidden"]))
        name = cls._own_name(prefix, params)
        if params.get("tied_to"):
            return [WeightSpec(name, shape, IGNORED, optional=True)]
        return [WeightSpec(name, shape, MATRIX)]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        src = self.params.get("tied_to") or self._own_name(self.prefix, self.params)
        self.linear = Linear(tensors[src])

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        """x [W, hidden] -> float32 logits [W, vocab]."""
        logits = self.linear.forward(x, out_dtype=torch.float32)
        if self.scale != 1.0:
            logits.mul_(self.scale)
        return ops.softcap(logits, self.softcap) if self.softcap else logits


register_part("embedding", "token_embedding", TokenEmbedding)
register_part("embedding", "sinusoid_norm_embedding", SinusoidNormEmbedding)
register_part("embedding", "bigram_embedding", BigramEmbedding)
register_part("lm_head", "linear_head", LinearHead)
