"""``general_delta``: linear attention by the generalized delta rule.  Per head, with r, k, v of ``dim`` each
(``r = W_r h`` and so on), a decay and a removal rate per key channel,

    w_t = exp(-e^(-1/2) * sigmoid(W_w2 tanh(W_w1 h_t) + w0))        in (exp(-e^(-1/2)), 1)
    a_t = sigmoid(W_a h_t + a_b)
    u_t = k_t / sqrt(sum(k_t^2) + 1e-6)                              the head's unit key
    S_t = diag(w_t) S_{t-1} - (a_t * u_t)(u_t^T S_{t-1}) + k_t v_t^T   S: [dim x dim], float32, zero at the start;
                                                                      the decay and the removal both read S_{t-1}
    o_t = S_t^T r_t

every head's o is divided by its root mean square, the heads side by side are multiplied by a weight over all of them
and by sigmoid(W_g h), and projected.  r, k, v, the raw removal rates, the gate and the decay's inner projection are
one stacked product whose sums stay float32; the decay, the removal rate, the unit key, the state and the norm are
float32 in either engine type.  The inner size of the decay's two-step projection is the stored tensors' own.  The
state lives in the request's state slot.

``gated_delta``: the gated delta rule.  Per head, with unit query and key (``kv_heads`` of them, shared by
``heads / kv_heads`` value heads each) and one decay and one rate per head and token,

    (q, k, v) = silu(conv(W_q h, W_k h, W_v h))                      a causal convolution over time on every channel
    q = q / sqrt(sum(q^2) + 1e-6) * dim^(-1/2),   k = k / sqrt(sum(k^2) + 1e-6)
    g_t = exp(-exp(A_log) softplus(W_a h_t + dt_bias)),   beta_t = sigmoid(W_b h_t)
    S <- g_t S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T     S: [dim x vdim], float32, zero at the start
    o_t = S^T q_t

every head's o is divided by its root mean square, multiplied by a weight ``vdim`` long that the heads share and by
silu(W_g h) (or sigmoid of it), and projected.  With ``decay`` ``channel`` there is one decay per head and key channel,

    g_t = exp(-exp(A_log) softplus(W_a2 W_a1 h_t + dt_bias))         heads x dim;   S <- diag(g_t) S

(A_log one a head).  The decays and, with ``two_step``, the gate (W_g2 W_g1 h) are projected in two steps: the two inner
products are rows of the stacked one, and both outer products are one product over the inner rows side by side.  All input projections are one stacked product whose sums stay float32, and so does
everything up to the output projection's input.  The state and the last ``taps - 1`` inputs of the convolutions live in
the request's state slot, so a prompt may be cut anywhere; a portion is cut into segments whose part that does not
depend on the state is worked out side by side.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, List

import torch

from ..config.registry import register_part
from ..kernels import ops
from ..weights.loader import MATRIX, VECTOR, WeightSpec
from .base import Part, RunInfo, StateNeed
from .linear import Linear
from .state_space import describe_row_entries

DECAY_SCALE = math.exp(-0.5)
KEY_EPS = 1e-6


class GeneralDelta(Part):
    """params: ``hidden``, ``heads``, ``dim``, ``decay_rank`` (0 = whatever the stored ``w1`` has), ``eps`` (of the
    per-head norm), ``decay_scale`` and ``key_eps`` (default ``e^(-1/2)`` and 1e-6), ``name`` (tensors
    ``<prefix>.<name>.{r,k,v,a,a.b,g,w1,w2,w0,norm,o}``).  State: ``delta`` float32 ``[heads, dim (value), dim (key)]``."""

    family = "mixer"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        p = params
        self.hidden, self.heads, self.dim = int(p["hidden"]), int(p["heads"]), int(p["dim"])
        self.eps = float(p["eps"])
        self.decay_scale = float(p.get("decay_scale", DECAY_SCALE))
        self.key_eps = float(p.get("key_eps", KEY_EPS))
        if not 1 <= self.dim <= 512:
            raise ValueError("general_delta: dim must be within 1..512")
        self.rank = 0
        self.stacked: Linear = None
        self.w2: Linear = None
        self.o: Linear = None

    @classmethod
    def weight_specs(cls, params: Dict[str, Any], prefix: str) -> List[WeightSpec]:
        h, hd = int(params["hidden"]), int(params["heads"]) * int(params["dim"])
        rank = int(params.get("decay_rank") or 0) or -1
        n = lambda leaf: cls.full_name(prefix, params, leaf)
        return ([WeightSpec(n(x), (hd, h), MATRIX) for x in ("r", "k", "v", "a", "g")]
                + [WeightSpec(n("a.b"), (hd,), VECTOR, std=0.5), WeightSpec(n("w1"), (rank, h), MATRIX),
                   WeightSpec(n("w2"), (hd, rank), MATRIX, std=0.5), WeightSpec(n("w0"), (hd,), VECTOR, std=0.5),
                   WeightSpec(n("norm"), (hd,), VECTOR, init="one_plus_normal"), WeightSpec(n("o"), (h, hd), MATRIX)])

    @classmethod
    def state_needs(cls, params: Dict[str, Any]) -> List[StateNeed]:
        d = int(params["dim"])
        return [StateNeed("delta", (int(params["heads"]), d, d), torch.float32)]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = lambda leaf: self.full_name(self.prefix, self.params, leaf)
        f32 = lambda leaf: tensors.pop(n(leaf)).to(torch.float32).contiguous()
        mats = [tensors.pop(n(x)) for x in ("r", "k", "v", "a", "g", "w1")]
        w2 = tensors.pop(n("w2"))
        self.rank = mats[-1].shape[0]
        if w2.shape[1] != self.rank:
            raise ValueError(f"{n('w2')} takes {w2.shape[1]} inputs but {n('w1')} gives {self.rank}")
        if len({m.dtype for m in mats}) > 1:
            mats = [m.float() for m in mats]
        self.stacked = Linear(torch.cat(mats, dim=0))
        del mats
        self.w2 = Linear(w2)
        self.a_bias, self.w0, self.norm_w = f32("a.b"), f32("w0"), f32("norm")
        self.o = Linear(tensors.pop(n("o")))

    @property
    def inner_width(self) -> int:
        return self.heads * self.dim

    def inner(self, x: torch.Tensor, ctx, run: RunInfo, position=None, out: torch.Tensor = None) -> torch.Tensor:
        """The normed, gated heads ``[N, heads * dim]`` that the output projection takes."""
        n, dev, hd = x.shape[0], x.device, self.heads * self.dim
        proj = self.stacked.forward(x, out_dtype=torch.float32)               # [r | k | v | a | g | w1]
        t = torch.empty((n, self.rank), dtype=x.dtype, device=dev)
        ops.activation(proj[:, 5 * hd:], t, ops.ACT_TANH)
        w_raw = self.w2.forward(t, out_dtype=torch.float32)
        o = torch.empty((n, hd), dtype=torch.float32, device=dev)
        ops.delta_rule_scan(proj, 0, hd, 2 * hd, 3 * hd, w_raw, self.w0, self.a_bias, run.states["delta"],
                            ctx.entry_q_start, ctx.entry_q_len, ctx.entry_slot, ctx.n_entries, o, self.heads, self.dim,
                            self.dim, self.decay_scale, self.key_eps)
        if out is None:
            out = torch.empty((n, hd), dtype=x.dtype, device=dev)
        return ops.head_norm_gate(o, proj[:, 4 * hd:5 * hd], self.norm_w, out, self.heads, self.dim, self.eps, ops.GATE_SIGMOID)

    def forward(self, x: torch.Tensor, ctx, run: RunInfo, position):
        return self.o.forward(self.inner(x, ctx, run), allow_partials=True, f32_sums=True, out_dtype=torch.float32)


register_part("mixer", "general_delta", GeneralDelta)


@dataclass
class GatedDeltaStep:
    """The entry of every row, and the step cut into segments for the scan kernels: int32 device tensors; ``n_segments``
    0 = every entry brings one token."""

    row_entry: torch.Tensor
    seg_entry: torch.Tensor
    seg_t0: torch.Tensor
    entry_first_seg: torch.Tensor
    n_segments: int


class GatedDelta(Part):
    """params: ``hidden``, ``heads``, ``kv_heads`` (default ``heads``), ``dim``, ``vdim``, ``conv`` (taps), ``eps`` (of the
    per-head norm), ``q_scale`` (default ``dim^-1/2``), ``key_eps`` (default 1e-6), ``decay`` (``head`` or ``channel``, the
    latter projected in two steps), ``gate`` (``silu`` or ``sigmoid``), ``two_step`` (the gate's projection), ``name`` (tensors
    ``<prefix>.<name>.{q,k,v,a,b,g,o,A_log,dt_bias,norm}`` and ``.{q,k,v}.conv`` ``[channels, taps]``; ``b`` is the rate's
    projection; a projection in two steps is ``{a1,a2}`` or ``{g1,g2}``, its inner size the stored tensors' own).  State: ``gated_delta`` float32 ``[heads, dim, vdim]``, ``gated_delta_tail`` float32 ``[taps - 1,
    channels of q, k and v]``."""

    family = "mixer"
    describe_key = "gated_delta_segments"

    def __init__(self, params, prefix, dtype, device):
        super().__init__(params, prefix, dtype, device)
        p = params
        self.hidden, self.heads = int(p["hidden"]), int(p["heads"])
        self.kv_heads = int(p.get("kv_heads") or p["heads"])
        self.dim, self.vdim, self.taps = int(p["dim"]), int(p["vdim"]), int(p["conv"])
        self.eps, self.key_eps = float(p["eps"]), float(p.get("key_eps", KEY_EPS))
        self.q_scale = float(p["q_scale"]) if p.get("q_scale") is not None else float(self.dim) ** -0.5
        if self.heads % self.kv_heads:
            raise ValueError(f"gated_delta: heads {self.heads} is not a multiple of kv_heads {self.kv_heads}")
        if not 1 <= self.dim <= 256:
            raise ValueError("gated_delta: dim must be within 1..256")
        if not 1 <= self.taps <= 16:
            raise ValueError("gated_delta: conv must be within 1..16 taps")
        self.by_channel = {"head": False, "channel": True}.get(p.get("decay", "head"))
        self.gate = {"silu": ops.GATE_SILU, "sigmoid": ops.GATE_SIGMOID}.get(p.get("gate", "silu"))
        if self.by_channel is None or self.gate is None:
            raise ValueError("gated_delta: decay is 'head' or 'channel', gate is 'silu' or 'sigmoid'")
        self.two_step = bool(p.get("two_step"))
        self.channels = self._channels(p)
        self.stacked: Linear = None         # [q; k; v; the one-step ones of g and a; the inner ones of a and g; b]
        self.outer: Linear = None           # the outer steps of a and g over the inner rows
        self.o: Linear = None

    @classmethod
    def _channels(cls, p) -> int:
        nk = int(p.get("kv_heads") or p["heads"])
        return 2 * nk * int(p["dim"]) + int(p["heads"]) * int(p["vdim"])

    @classmethod
    def weight_specs(cls, params: Dict[str, Any], prefix: str) -> List[WeightSpec]:
        h, nh, d, vd, taps = (int(params[k]) for k in ("hidden", "heads", "dim", "vdim", "conv"))
        nk = int(params.get("kv_heads") or nh)
        n = lambda leaf: cls.full_name(prefix, params, leaf)
        rows = {"q": nk * d, "k": nk * d, "v": nh * vd}
        return ([WeightSpec(n(x), (r, h), MATRIX) for x, r in rows.items()]
                + [WeightSpec(n(f"{x}.conv"), (r, taps), VECTOR, std=0.5) for x, r in rows.items()]
                + cls._projection(params, n, "g", params.get("two_step"), nh * vd, h)
                + cls._projection(params, n, "a", params.get("decay") == "channel", nh * d if params.get("decay") == "channel" else nh, h)
                + [WeightSpec(n("b"), (nh, h), MATRIX), WeightSpec(n("A_log"), (nh,), VECTOR, std=0.5),
                   WeightSpec(n("dt_bias"), (nh * d if params.get("decay") == "channel" else nh,), VECTOR, std=0.5),
                   WeightSpec(n("norm"), (vd,), VECTOR, init="one_plus_normal"), WeightSpec(n("o"), (h, nh * vd), MATRIX)])

    @staticmethod
    def _projection(params, n, leaf: str, two_step: bool, rows: int, hidden: int) -> List[WeightSpec]:
        if not two_step:
            return [WeightSpec(n(leaf), (rows, hidden), MATRIX)]
        rank = int(params.get("rank") or 128)              # of random weights; stored ones have their own
        return [WeightSpec(n(leaf + "1"), (-1, hidden), MATRIX, free_size=rank),
                WeightSpec(n(leaf + "2"), (rows, -1), MATRIX, std=rank ** -0.5, free_size=rank)]

    @classmethod
    def state_needs(cls, params: Dict[str, Any]) -> List[StateNeed]:
        needs = [StateNeed("gated_delta", (int(params["heads"]), int(params["dim"]), int(params["vdim"])), torch.float32)]
        if int(params["conv"]) > 1:
            needs.append(StateNeed("gated_delta_tail", (int(params["conv"]) - 1, cls._channels(params)), torch.float32))
        return needs

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = lambda leaf: self.full_name(self.prefix, self.params, leaf)
        f32 = lambda leaf: tensors.pop(n(leaf)).to(torch.float32).contiguous()
        mats = {x: tensors.pop(n(x)) for x in (["q", "k", "v"] + ([] if self.two_step else ["g"]) + ([] if self.by_channel else ["a"]))}
        outer = []                                         # (second step, its inner size), the decays' first
        for leaf, on in (("a", self.by_channel), ("g", self.two_step)):
            if on:
                mats[leaf + "1"], second = tensors.pop(n(leaf + "1")), tensors.pop(n(leaf + "2"))
                if second.shape[1] != mats[leaf + "1"].shape[0]:
                    raise ValueError(f"{n(leaf + '2')} takes {second.shape[1]} inputs but {n(leaf + '1')} gives {mats[leaf + '1'].shape[0]}")
                outer.append(second)
        mats["b"] = tensors.pop(n("b"))
        if len({m.dtype for m in (*mats.values(), *outer)}) > 1:
            mats, outer = {k: m.float() for k, m in mats.items()}, [m.float() for m in outer]
        self.inner_cols = -(-sum(m.shape[1] for m in outer) // 8) * 8          # rows of zeros fill the inner ones up to eights
        if outer:
            like = mats["b"]
            fill = like.new_zeros((self.inner_cols - sum(m.shape[1] for m in outer), self.hidden))
            b = mats.pop("b")
            mats.update(fill=fill, b=b)
            joint, row, col = like.new_zeros((sum(m.shape[0] for m in outer), self.inner_cols)), 0, 0
            for m in outer:
                joint[row:row + m.shape[0], col:col + m.shape[1]] = m
                row, col = row + m.shape[0], col + m.shape[1]
            self.outer = Linear(joint)
        self.at, row = {}, 0                               # where each block of the stacked product begins
        for k, m in mats.items():
            self.at[k], row = row, row + m.shape[0]
        self.at["inner"] = self.at.get("a1", self.at.get("g1", 0))
        if outer and row % 4:                              # rows of float32 sums that start on 16-byte boundaries
            mats["end"] = mats["b"].new_zeros((4 - row % 4, self.hidden))
        self.stacked = Linear(torch.cat(list(mats.values()), dim=0))
        del mats, outer
        self.conv_w = torch.cat([f32(f"{x}.conv") for x in ("q", "k", "v")]).contiguous()
        self.a_log, self.dt_bias = f32("A_log"), f32("dt_bias")
        self.norm_w = f32("norm").repeat(self.heads).contiguous()
        self.o = Linear(tensors.pop(n("o")))

    def describe_step(self, layout, put) -> GatedDeltaStep:
        rows = describe_row_entries(layout, put)
        lens = [int(v) for v in layout.q_len[:layout.n_entries]]
        if all(v == 1 for v in lens):
            return GatedDeltaStep(rows, put([]), put([]), put([]), 0)
        seg = ops.gated_delta_segment() if torch.device(self.device).type == "cuda" else 32
        seg_entry, seg_t0, first = [], [], []
        for i, v in enumerate(lens):
            first.append(len(seg_entry))
            for t0 in range(0, v, seg):
                seg_entry.append(i), seg_t0.append(t0)
        return GatedDeltaStep(rows, put(seg_entry), put(seg_t0), put(first), len(seg_entry))

    @property
    def inner_width(self) -> int:
        return self.heads * self.vdim

    def inner(self, x: torch.Tensor, ctx, run: RunInfo, position=None, out: torch.Tensor = None) -> torch.Tensor:
        """The normed, gated heads ``[N, heads * vdim]`` that the output projection takes."""
        n, dev = x.shape[0], x.device
        kd, hv, c = self.kv_heads * self.dim, self.heads * self.vdim, self.channels
        step: GatedDeltaStep = ctx.extras[self.describe_key]
        proj = self.stacked.forward(x, out_dtype=torch.float32)
        outer = None                                       # [decays | gate] of what is projected in two steps
        if self.outer is not None:
            rows = torch.empty((n, self.inner_cols), dtype=x.dtype, device=dev)
            ops.activation(proj[:, self.at["inner"]:self.at["inner"] + self.inner_cols], rows, ops.ACT_NONE)
            outer = self.outer.forward(rows, out_dtype=torch.float32)
        decay = outer[:, :self.heads * self.dim] if self.by_channel else None
        gate = outer[:, outer.shape[1] - hv:] if self.two_step else proj[:, self.at["g"]:self.at["g"] + hv]
        qkv = torch.empty((n, c), dtype=torch.float32, device=dev)
        ops.causal_conv_heads(proj, 0, c, self.conv_w, None, run.states["gated_delta_tail"] if self.taps > 1 else None,
                              step.row_entry, ctx.entry_q_start, ctx.entry_q_len, ctx.entry_slot, ctx.n_entries, qkv,
                              2 * self.kv_heads, self.dim, self.kv_heads, self.q_scale, self.key_eps)
        o = torch.empty((n, hv), dtype=torch.float32, device=dev)
        ops.gated_delta_scan(qkv, 0, kd, 2 * kd, proj, self.at.get("a", 0), self.at["b"], self.a_log, self.dt_bias,
                             run.states["gated_delta"], ctx.entry_q_start, ctx.entry_q_len, ctx.entry_slot, ctx.n_entries, o,
                             self.heads, self.kv_heads, self.dim, self.vdim, step.seg_entry, step.seg_t0, step.entry_first_seg,
                             step.n_segments, decay)
        if out is None:
            out = torch.empty((n, hv), dtype=x.dtype, device=dev)
        return ops.head_norm_gate(o, gate, self.norm_w, out, self.heads, self.vdim, self.eps, self.gate)

    def forward(self, x: torch.Tensor, ctx, run: RunInfo, position):
        return self.o.forward(self.inner(x, ctx, run), allow_partials=True, f32_sums=True, out_dtype=torch.float32)


register_part("mixer", "gated_delta", GatedDelta)
