"""Parts that rewrite the stream between layers (family ``junction``).

``loop_entry``: where a pass over a stretch of layers begins, the stream is
renewed from itself and from the embedding output,

    x <- W_in [x ; x0] + step[t]          W_in [hidden, 2 hidden], step [passes, hidden]

``t`` being the number of the pass (the run's parameter ``pass``) and ``x0``
the stream as the embedding left it.  The half of the product that reads x0
is the same in every pass and is made once per step; the sum is float32.

``add_embedding``: ``x <- x + x0``, nothing else.

``loop_step``: ``x <- x + x0 + step[t]``, without ``x0`` ahead of the first
pass.  It rewrites nothing itself: it hands what it adds on with the pending
sum, and the norm that comes next adds it all.

``stream_join``: how a sublayer's result joins a stream of several copies; like
``loop_step`` it only says what is to be done, and the norm that comes next
does it.
"""
from __future__ import annotations

from typing import Any, Dict, List

import torch

from ..config.registry import register_part
from ..kernels import ops
from ..weights.loader import MATRIX, VECTOR, WeightSpec
from .base import JoinedSum, Part, RunInfo, StreamMix
from .linear import Linear


class LoopEntry(Part):
    """params: ``hidden``, ``passes``, ``in_name``, ``step_name`` (full tensor names)."""

    family = "junction"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.hidden, self.passes = int(params["hidden"]), int(params["passes"])
        self.from_x: Linear = None
        self.from_x0: Linear = None
        self.step: torch.Tensor = None

    @classmethod
    def weight_specs(cls, params: Dict[str, Any], prefix: str) -> List[WeightSpec]:
        h, t = int(params["hidden"]), int(params["passes"])
        return [WeightSpec(params["in_name"], (h, 2 * h), MATRIX, std=0.7 / h ** 0.5),
                WeightSpec(params["step_name"], (t, h), VECTOR)]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        w = tensors.pop(self.params["in_name"])
        self.from_x = Linear(w[:, :self.hidden].contiguous())
        self.from_x0 = Linear(w[:, self.hidden:].contiguous())
        self.step = tensors.pop(self.params["step_name"]).to(torch.float32).contiguous()

    def _operand(self, t: torch.Tensor) -> torch.Tensor:
        if self.dtype == torch.float32:
            return t
        return ops.convert(t, torch.empty(t.shape, dtype=self.dtype, device=t.device))

    def forward(self, residual: torch.Tensor, ctx, run: RunInfo) -> None:
        key = ("loop_entry", id(self))
        base = ctx.scratch.get(key)
        if base is None:
            base = ctx.scratch[key] = self.from_x0.forward(self._operand(ctx.embedding_output), out_dtype=torch.float32)
        y = self.from_x.forward(self._operand(residual), out_dtype=torch.float32)
        ops.add_rows_vector(y, base, self.step[int(run.params["pass"])], residual)


class AddEmbedding(Part):
    """``x <- x + x0`` with ``x0`` the stream as the embedding left it: where a later pass over a stretch of layers
    begins, the tokens' embeddings join the stream again.  No weights; params: none."""

    family = "junction"

    def forward(self, residual: torch.Tensor, ctx, run: RunInfo) -> None:
        ops.add_into(residual, ctx.embedding_output, 1)


class LoopStep(Part):
    """What joins the stream ahead of pass ``t`` (the run's parameter ``pass``) over a stretch of layers: the vector
    ``step[t]`` and, from the second pass on, the stream as the embedding left it.  params: ``hidden``, ``passes``,
    ``step_name`` (the full name of the tensor ``[passes, hidden]``)."""

    family = "junction"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.hidden, self.passes = int(params["hidden"]), int(params["passes"])
        self.step: torch.Tensor = None

    @classmethod
    def weight_specs(cls, params: Dict[str, Any], prefix: str) -> List[WeightSpec]:
        return [WeightSpec(params["step_name"], (int(params["passes"]), int(params["hidden"])), VECTOR, std=0.3)]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.step = tensors.pop(self.params["step_name"]).to(torch.float32).contiguous()

    def pending(self, delta, ctx, run: RunInfo) -> JoinedSum:
        t = int(run.params["pass"])
        return JoinedSum(delta, ctx.embedding_output if t > 0 else None, self.step[t])


class StreamJoin(Part):
    """``X_t <- sum_s mix[s, t] X_s + factor * out[t] * y`` for a sublayer's result ``y`` and the stream's copies ``X_s``.
    params: ``streams``, ``factor`` (default 1; it joins ``out`` at load, in float32), ``name`` (tensors
    ``<prefix>.<name>.mix`` ``[streams, streams]`` and ``.out`` ``[streams]``)."""

    family = "junction"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.streams, self.factor = int(params["streams"]), float(params.get("factor", 1.0))
        self.mix: torch.Tensor = None
        self.out: torch.Tensor = None

    @classmethod
    def weight_specs(cls, params: Dict[str, Any], prefix: str) -> List[WeightSpec]:
        s = int(params["streams"])
        return [WeightSpec(cls.full_name(prefix, params, "mix"), (s, s), VECTOR, std=s ** -0.5),
                WeightSpec(cls.full_name(prefix, params, "out"), (s,), VECTOR, init="one_plus_normal", std=0.1)]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        f32 = lambda leaf: tensors.pop(self.full_name(self.prefix, self.params, leaf)).to(torch.float32)
        self.mix = f32("mix").contiguous()
        self.out = (f32("out") * self.factor).contiguous()

    def pending(self, delta, ctx, run: RunInfo) -> StreamMix:
        return StreamMix(delta, self.mix, self.out)


register_part("junction", "stream_join", StreamJoin)
register_part("junction", "loop_entry", LoopEntry)
register_part("junction", "loop_step", LoopStep)
register_part("junction", "add_embedding", AddEmbedding)
