"""What every part has in common, and what a mixer may ask of the cache.

A part is built from its :class:`~inferflux_b200.config.spec.PartSpec`
parameters alone: it never sees the architecture's name or configuration.  It
declares the tensors it wants (:meth:`Part.weight_specs`), receives them once
(:meth:`Part.load`, where it may fuse or re-lay them), and is then called by
the step function.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

import torch

from ..weights.loader import WeightSpec


@dataclass(frozen=True)
class CacheStream:
    """One tensor that a mixer keeps per token in the paged cache: ``heads``
    vectors of ``width`` elements.  Within a page a stream lies as
    ``[head][slot][width]``, so one head's vectors of a page are contiguous."""

    name: str
    heads: int
    width: int


@dataclass(frozen=True)
class KVNeed:
    """What a mixer keeps per token in pages: one or more streams (keys and
    values for attention; a single latent vector for a mixer that caches
    one), and for how long: ``window`` None = every token is kept, w = only
    the last w; ``chunk`` c = only those of the newest token's stretch of c
    positions.  Runs whose mixers ask for equal needs share a cache group."""

    streams: Tuple[CacheStream, ...]
    window: Optional[int] = None
    keep_first: int = 0         # with a window: this many first tokens stay visible (and cached) for good
    chunk: Optional[int] = None # tokens see their own chunk of so many positions only (counted from the sequence's start)

    @classmethod
    def keys_and_values(cls, n_kv_heads: int, head_dim: int, window: Optional[int] = None,
                        value_dim: Optional[int] = None, keep_first: int = 0, chunk: Optional[int] = None) -> "KVNeed":
        """``n_kv_heads * head_dim`` keys and as many values per token (values ``value_dim`` wide if given)."""
        return cls((CacheStream("k", n_kv_heads, head_dim), CacheStream("v", n_kv_heads, value_dim or head_dim)),
                   window, keep_first if window else 0, chunk)

    @property
    def elements_per_token(self) -> int:
        return sum(s.heads * s.width for s in self.streams)


@dataclass(frozen=True)
class StateNeed:
    """Per-request state of fixed size, kept in the request's state slot."""

    name: str
    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


class PartialSums:
    """A value given as float32 slices ``[S, N, H]`` whose sum it is.  A mixer
    or feed-forward may return one instead of a tensor; the norm that follows
    adds the slices (in index order) while it adds the residual."""

    def __init__(self, tensor: torch.Tensor):
        self.tensor = tensor
        self.count = tensor.shape[0]


class BranchMean:
    """A mixer's result given as the mean of branches, each the float32 sums of one branch (a tensor or
    :class:`PartialSums`) normed with a weight of its own: ``(N(a) * w_a + N(b) * w_b) / 2`` with
    ``N(v) = v / sqrt(mean(v^2) + eps)``.  The norm that takes it computes it while it adds."""

    def __init__(self, branches, eps: float):
        self.branches = list(branches)          # [(sums, weight float32 [H]), ...]: two of them
        self.eps = eps


class ScaledSum:
    """A mixer's result given as a weighted sum of branches, ``s_a * a + s_b * b``, each branch the float32 sums of
    one mixer (a tensor or :class:`PartialSums`).  The norm that takes it computes the sum while it adds to the stream."""

    def __init__(self, terms):
        self.terms = list(terms)                # [(sums, factor), ...]: two of them


class JoinedSum:
    """A pending result that is joined by rows of its own and one vector for all rows: ``value + rows + vector``, with
    ``value`` a tensor, :class:`PartialSums`, :class:`ScaledSum` or None, ``rows`` float32 ``[N, H]`` or None and
    ``vector`` float32 ``[H]`` or None.  What a junction adds to the stream goes on like this, so that the next norm
    adds everything in one pass."""

    def __init__(self, value, rows: Optional[torch.Tensor], vector: Optional[torch.Tensor]):
        self.value, self.rows, self.vector = value, rows, vector


class StreamMix:
    """A sublayer's result on its way into a stream of several copies: ``X_t <- sum_s mix[s, t] X_s + out[t] * value``,
    all copies at once from the old ones; ``value`` a tensor or :class:`PartialSums`, ``mix`` float32 ``[S, S]`` (from, to),
    ``out`` float32 ``[S]``.  The norm that comes next mixes the copies while it reads them."""

    def __init__(self, value, mix: torch.Tensor, out: torch.Tensor):
        self.value, self.mix, self.out = value, mix, out


class NormedDelta:
    """A sublayer's result that is to be normed before it joins the stream: ``N(value) * weight`` with ``value``
    a tensor, :class:`PartialSums` or :class:`BranchMean`.  Blocks with a norm behind every sublayer hand this
    to the next norm, which does both norms and the sum in one pass over the row."""

    def __init__(self, value, weight: torch.Tensor, eps: float):
        self.value, self.weight, self.eps = value, weight, eps


class Part:
    """Base of all parts.  ``params`` are the PartSpec's parameters, ``prefix``
    the weight-name prefix of the enclosing layer ("" at model level).

    Interfaces by family (``x`` = ``[N, hidden]`` rows of the step's flattened
    tokens, ``ctx`` = the step's :class:`~inferflux_b200.engine.batch.StepContext`):

    * ``mixer``: ``forward(x, ctx, run, position) -> Tensor | PartialSums``.
      ``run`` is the :class:`RunInfo` of this execution of the layer (its cache
      group and index, its state tensors); ``position`` is whatever the position
      encoding named by the layer returned from ``prepare`` for this step, or
      None.
    * ``feed_forward``: ``forward(x, ctx) -> Tensor | PartialSums``.
    * ``norm``: ``forward(residual, delta, out=None, rows=None) -> Tensor``:
      adds ``delta`` (tensor, PartialSums or None) into the float32 residual
      unless ``rows`` selects rows, returns the normed rows.
    * ``position``: ``prepare(ctx) -> object``, once per step for all layers.
      The contract between a position encoding and the mixers that consume it
      is the type of that object.  The built-in ``gqa_attention`` takes a pair
      ``(cos, sin)`` of float32 ``[N, r/2]`` tensors, ``r <= head_dim`` even,
      and rotates the first ``r`` dimensions of every query and key head in
      split-half pairs ``(i, i + r/2)``; any position part that returns such a
      pair serves it.  A mixer with another idea of position defines its own
      object and says so in its docstring.
    * ``embedding``: ``forward_step(ctx) -> float32 [N, hidden]`` (the default
      calls ``forward(token_ids)``; one that adds positions reads them from
      ``ctx``; one for a stream of several copies gives ``[N, copies, hidden]``,
      and its :meth:`state_needs` are tensors it finds in ``self.states``); ``lm_head``: ``forward(x) -> float32 [rows, vocab]``.
    * ``shift``: ``forward(h32, ctx, run) -> Tensor``: mixes every row of the
      float32 normed rows with the row before it (the request's state slot
      holds the last row of the step before).
    * ``junction``: ``forward(residual, ctx, run) -> None``: rewrites the
      float32 stream in place between layers (a loop's entry, say).

    Any part may describe the step for its kernels (:meth:`describe_step`).  A part that is made of other
    parts (two mixers side by side, say) lists them in :meth:`subparts`; the model asks those for their
    descriptions too.
    """

    family = ""

    def __init__(self, params: Dict[str, Any], prefix: str, dtype: torch.dtype, device: str):
        self.params = dict(params)
        self.prefix = prefix
        self.dtype = dtype
        self.device = device

    def subparts(self) -> list:
        return []

    # -- naming ---------------------------------------------------------
    @staticmethod
    def full_name(prefix: str, params: Dict[str, Any], leaf: str = "") -> str:
        parts = [p for p in (prefix, params.get("name", ""), leaf) if p]
        return ".".join(parts)

    # -- weights --------------------------------------------------------
    @classmethod
    def weight_specs(cls, params: Dict[str, Any], prefix: str) -> List[WeightSpec]:
        return []

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Take the tensors named by :meth:`weight_specs` (those that exist)."""

    # -- cache ----------------------------------------------------------
    @classmethod
    def kv_need(cls, params: Dict[str, Any]) -> Optional[KVNeed]:
        return None

    @classmethod
    def state_needs(cls, params: Dict[str, Any]) -> List[StateNeed]:
        return []

    # -- the step -------------------------------------------------------
    #: Parts with the same key share one description per step (the key names the
    #: kind of description, e.g. the tile lists of one family of kernels); None =
    #: the part needs none.
    describe_key: Optional[str] = None

    def describe_step(self, layout, put) -> object:
        """Per-step metadata for this part's kernels, derived on the host from
        ``layout`` (:class:`~inferflux_b200.engine.batch.StepLayout`: how many
        tokens each entry brings and how many it has cached).  ``put(values)``
        appends int32 values to the step's metadata (one host-to-device copy for
        the whole step) and returns their device view.  The result is kept in
        ``ctx.extras[describe_key]``.  Called once per step and key, before the
        copy; in a captured step of single tokens the copy is repeated with new
        token ids, positions and block tables only, so what this writes for such
        a step may depend on the number of entries and on :meth:`step_shape`
        alone."""
        return None

    def step_shape(self, layout) -> tuple:
        """What, beyond the number of entries and the width of the block tables,
        decides which kernels this part launches in a step of single tokens (it
        becomes part of the key under which such steps are captured)."""
        return ()


@dataclass
class RunInfo:
    """Where one run of a layer finds its cache.

    kv_group / kv_index: the cache group and the run's place in it (None for a
    mixer without paged keys and values); writes_kv False = reads another
    run's cache.  states: the run's per-request state tensors
    ``[max_seqs, *shape]`` by name.  params: the run's own parameters from
    the schedule (:class:`~inferflux_b200.config.spec.Run`)."""

    run_index: int
    kv_group: Optional[int] = None
    kv_index: Optional[int] = None
    writes_kv: bool = True
    states: Optional[Dict[str, torch.Tensor]] = None
    params: Optional[Dict[str, Any]] = None
