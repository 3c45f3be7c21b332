"""Root-mean-square norm fused with the residual sum.

``residual += delta;  out = residual * rsqrt(mean(residual^2) + eps) * weight``
in float32 on the float32 residual stream, rounded once on output
(reference: runtime/backends/cuda/native/cuda_kernels.cu:469-501 norm,
:541-579 fused add + norm; call sites
runtime/backends/cuda/native/transformer_forward.cu:1413-1424,1744-1754).
"""
from __future__ import annotations

from typing import Any, Dict, List, Optional

import torch

from ..config.registry import register_part
from ..kernels import ops
from ..weights.loader import VECTOR, WeightSpec
from .base import BranchMean, JoinedSum, NormedDelta, Part, PartialSums, ScaledSum, StreamMix


class RMSNorm(Part):
    """params: ``hidden``, ``eps``, and the weight's name: ``name`` (weight is ``<prefix>.<name>.weight``) or
    ``weight_name`` (the leaf itself, ``<prefix>.<weight_name>``); ``weight_offset`` (default 0) joins the stored weight
    at load, in float32 (1 for a weight that is stored around zero).

    ``delta`` may also be a :class:`NormedDelta` (a sublayer's result that is normed before it joins the
    stream, itself possibly the mean of two normed branches): both norms and the sum are one kernel."""

    family = "norm"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.hidden = int(params["hidden"])
        self.eps = float(params["eps"])
        self.weight: Optional[torch.Tensor] = None

    @classmethod
    def _weight_name(cls, prefix, params) -> str:
        if params.get("weight_name"):
            return ".".join(p for p in (prefix, params["weight_name"]) if p)
        return cls.full_name(prefix, params, "weight")

    @classmethod
    def weight_specs(cls, params: Dict[str, Any], prefix: str) -> List[WeightSpec]:
        if params.get("weight_offset"):
            return [WeightSpec(cls._weight_name(prefix, params), (int(params["hidden"]),), VECTOR, std=0.1)]
        return [WeightSpec(cls._weight_name(prefix, params), (int(params["hidden"]),), VECTOR, init="one_plus_normal")]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors[self._weight_name(self.prefix, self.params)].to(torch.float32).contiguous()
        if self.params.get("weight_offset"):
            self.weight = self.weight + float(self.params["weight_offset"])

    def forward(self, residual: torch.Tensor, delta, out: Optional[torch.Tensor] = None,
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Adds ``delta`` (a tensor, a :class:`PartialSums` or None) into the
        float32 ``residual`` (unless ``rows`` picks rows, which leaves it
        untouched) and returns the normed rows in the engine's type."""
        n_partials = 1
        n_rows = rows.numel() if rows is not None else residual.shape[0]
        if out is None:
            out = torch.empty((n_rows, self.hidden), dtype=self.dtype, device=residual.device)
        if isinstance(delta, NormedDelta):
            return normed_sum(residual, delta, self.weight, out, rows)
        if isinstance(delta, PartialSums):
            delta, n_partials = delta.tensor, delta.count
        return ops.add_rmsnorm(residual, delta, self.weight, self.eps, out, rows, n_partials)


def _sums(v) -> torch.Tensor:
    """float32 sums as the chain kernel takes them: ``[N, H]`` or slices ``[P, N, H]``."""
    if isinstance(v, PartialSums):
        return v.tensor
    if v.dtype != torch.float32:
        raise TypeError("a normed delta is made of float32 sums; a part gave " + str(v.dtype))
    return v


def normed_sum(residual: torch.Tensor, delta: NormedDelta, w_next: Optional[torch.Tensor], out: Optional[torch.Tensor],
               rows: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """``residual += N(value) * delta.weight`` and, with ``w_next``, ``out = N(residual) * w_next``, in one kernel;
    ``value`` may be the mean of two normed branches."""
    v = delta.value
    if isinstance(v, BranchMean):
        if len(v.branches) != 2:
            raise ValueError("the mean of normed branches is built for two branches")
        (a, wa), (b, wb) = v.branches
        return ops.norm_chain(residual, _sums(a), delta.eps, w_a=wa, b=_sums(b), w_b=wb, w_post=delta.weight,
                              w_next=w_next, out=out, rows=rows)
    return ops.norm_chain(residual, _sums(v), delta.eps, w_post=delta.weight, w_next=w_next, out=out, rows=rows)


class LayerNorm(Part):
    """Layer norm with a weight and no bias, fused with the residual sum:
    ``residual += delta;  out = (r - mean(r)) / sqrt(mean((r - mean(r))^2) + eps) * weight``
    in float32.  params: ``hidden``, ``eps``, and the weight's name: ``name``
    (weight is ``<prefix>.<name>.weight``) or ``weight_name`` (the leaf itself,
    ``<prefix>.<weight_name>``)."""

    family = "norm"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.hidden = int(params["hidden"])
        self.eps = float(params["eps"])
        self.weight: Optional[torch.Tensor] = None

    @classmethod
    def _weight_name(cls, prefix, params) -> str:
        if params.get("weight_name"):
            return ".".join(p for p in (prefix, params["weight_name"]) if p)
        return cls.full_name(prefix, params, "weight")

    @classmethod
    def weight_specs(cls, params: Dict[str, Any], prefix: str) -> List[WeightSpec]:
        return [WeightSpec(cls._weight_name(prefix, params), (int(params["hidden"]),), VECTOR, init="one_plus_normal")]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors[self._weight_name(self.prefix, self.params)].to(torch.float32).contiguous()

    def forward(self, residual: torch.Tensor, delta, out: Optional[torch.Tensor] = None,
                rows: Optional[torch.Tensor] = None, out32: Optional[torch.Tensor] = None) -> torch.Tensor:
        """As :meth:`RMSNorm.forward`; ``out32`` (float32 ``[rows, hidden]``)
        takes the normed rows unrounded as well."""
        n_partials = 1
        if isinstance(delta, PartialSums):
            delta, n_partials = delta.tensor, delta.count
        n_rows = rows.numel() if rows is not None else residual.shape[0]
        if out is None:
            out = torch.empty((n_rows, self.hidden), dtype=self.dtype, device=residual.device)
        return ops.add_layernorm(residual, delta, self.weight, self.eps, out, rows, n_partials, out32)


class GroupRMSNorm(RMSNorm):
    """RMS norm over ``groups`` equal consecutive parts of the row, each divided by its own root mean square, the whole
    multiplied by one weight of the row's length; fused with the sum into the stream like :class:`RMSNorm`.
    ``delta`` may also be a :class:`ScaledSum` of two branches, or a :class:`JoinedSum`: the weighted sum, what joins it,
    the sum into the stream and the norm are one kernel.  params: those of ``rmsnorm`` and ``groups`` (default 1, which is the plain norm)."""

    family = "norm"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.groups = int(params.get("groups") or 1)
        if self.groups < 1 or self.hidden % self.groups:
            raise ValueError(f"group_rmsnorm: {self.groups} groups do not divide a row of {self.hidden}")

    def forward(self, residual: torch.Tensor, delta, out: Optional[torch.Tensor] = None,
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        n_rows = rows.numel() if rows is not None else residual.shape[0]
        if out is None:
            out = torch.empty((n_rows, self.hidden), dtype=self.dtype, device=residual.device)
        if isinstance(delta, NormedDelta) or isinstance(delta, BranchMean):
            raise TypeError("group_rmsnorm takes a tensor, partial sums or a weighted sum of two branches")
        x = vec = None
        if isinstance(delta, JoinedSum):
            delta, x, vec = delta.value, delta.rows, delta.vector
        terms = delta.terms if isinstance(delta, ScaledSum) else ([(delta, 1.0)] if delta is not None else [])
        if len(terms) > 2:
            raise ValueError("a weighted sum is built for two branches")
        flat = [((v.tensor if isinstance(v, PartialSums) else v), float(f)) for v, f in terms] + [(None, 1.0)] * (2 - len(terms))
        (a, fa), (b, fb) = flat
        if rows is not None and any(t is not None for t in (a, b, x, vec)):
            # picked rows leave the stream untouched: the pending sum goes in first
            ops.add_group_rmsnorm(residual, a, self.weight, self.eps, self.groups, None, None, fa, b, fb, x, vec)
            a = b = x = vec = None
        return ops.add_group_rmsnorm(residual, a, self.weight, self.eps, self.groups, out, rows, fa, b, fb, x, vec)


class StreamRMSNorm(RMSNorm):
    """RMS norm of a weighted sum of the stream's copies, fused with what is pending for them: with ``X`` float32
    ``[N, streams, hidden]`` and a :class:`StreamMix` pending,

        X_t <- sum_s mix[s, t] X_s + out[t] * value;   u = sum_s reads[s] X_s;   result = u / sqrt(mean(u^2) + eps) * weight

    in one pass over the row.  params: those of ``rmsnorm``, ``streams``, and ``reads``: the leaf name of the weights
    ``[streams]`` (None = ones: the plain sum)."""

    family = "norm"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        self.streams = int(params["streams"])
        if not 1 <= self.streams <= ops.MAX_STREAMS:
            raise ValueError(f"stream_rmsnorm: {self.streams} streams are not within 1..{ops.MAX_STREAMS}")
        self.reads: Optional[torch.Tensor] = None

    @classmethod
    def weight_specs(cls, params: Dict[str, Any], prefix: str) -> List[WeightSpec]:
        specs = super().weight_specs(params, prefix)
        if params.get("reads"):
            specs.append(WeightSpec(cls.full_name(prefix, {}, params["reads"]), (int(params["streams"]),), VECTOR, std=0.5))
        return specs

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        super().load(tensors)
        if self.params.get("reads"):
            self.reads = tensors.pop(self.full_name(self.prefix, {}, self.params["reads"])).to(torch.float32).contiguous()
        else:
            self.reads = torch.ones(self.streams, dtype=torch.float32, device=self.weight.device)

    def forward(self, residual: torch.Tensor, delta, out: Optional[torch.Tensor] = None,
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        n_rows = rows.numel() if rows is not None else residual.shape[0]
        if out is None:
            out = torch.empty((n_rows, self.hidden), dtype=self.dtype, device=residual.device)
        value = mix = out_w = None
        if delta is not None:
            if not isinstance(delta, StreamMix):
                raise TypeError("stream_rmsnorm takes what a stream_join made of a sublayer's result")
            value, mix, out_w = delta.value, delta.mix, delta.out
            value = value.tensor if isinstance(value, PartialSums) else value
        return ops.stream_mix_norm(residual, value, mix, out_w, self.reads, self.weight, self.eps, out, rows)


register_part("norm", "stream_rmsnorm", StreamRMSNorm)
register_part("norm", "rmsnorm", RMSNorm)
register_part("norm", "group_rmsnorm", GroupRMSNorm)
register_part("norm", "layernorm", LayerNorm)
