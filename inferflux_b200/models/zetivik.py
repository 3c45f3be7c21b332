"""``Zetivik`` as a spec: the one file that knows this architecture.

A plain token embedding; every layer a ``prenorm`` block whose norms store their weight's distance from one.  A layer's
mixer is ``side_by_side`` with ``combine="weighted"``: ``window_attention`` inside chunks (biases on q, k and v, every
query and key head normed and rotated, one gate a head) beside ``gated_delta``, summed with the two factors the
configuration gives; or it is ``retention`` in its lightning form (silu on q, k and v, no rotation and no further
scale, all heads normed together, a sigmoid gate).  The feed-forward is ``clamped_glu`` without biases, or absent.  A
stretch of layers may run several times in a row on the same weights, every pass with caches and states of its own;
ahead of every pass a ``loop_step`` junction adds the pass's vector and, from the second on, the embedding's output.  A
last norm and an output head that is the embedding table, its logits capped.  Every distinct set of rotary parameters
is one position table, shared by the layers that use it.  Tensor names: ``embed``, ``loop.step``, ``l<i>.{norm1,norm2}``,
``l<i>.mix.{left,right}.*`` or ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``.
"""
from __future__ import annotations

import json

from ..config.model_config import ConfigError, ZetivikConfig
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, Run

MAX_POSITION = 1 << 20      # the design has no longest sequence; this bounds the engine's bookkeeping
GLU_ALPHA, GLU_SHIFT = 1.702, 1.0       # the feed-forward's two constants: g * sigmoid(1.702 g) * (u + 1)


def build_zetivik_spec(cfg: ZetivikConfig) -> ModelSpec:
    h, eps = cfg.width, cfg.norm_eps
    positions, by_params = {}, {}

    def position_of(rot) -> str:
        """The name of the table for these rotary parameters (None if nothing rotates)."""
        if not rot["dims"]:
            return None
        key = json.dumps(rot, sort_keys=True)
        if key not in by_params:
            by_params[key] = f"rot{len(by_params)}"
            positions[by_params[key]] = PartSpec("rotary", dict(rotary_dim=rot["dims"], theta=rot["base"]))
        return by_params[key]

    norm = lambda leaf: PartSpec("group_rmsnorm", dict(weight_name=leaf, hidden=h, eps=eps, groups=1, weight_offset=1.0))
    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        if layer.type == "parallel":
            l, r = m["left"], m["right"]
            left = dict(kind="window_attention", position=position_of(l["rot"]), out=None, params=dict(
                name="mix.left", hidden=h, heads=l["heads"], kv_heads=l["kv_heads"], dim=l["dim"], vdim=l["vdim"], conv=0,
                rot_dims=l["rot"]["dims"], rot_layout="half", scale=l["scale"], softcap=None, window=None, chunk=l["chunk"],
                sink=False, gate="heads", qk_norm="heads", bias="qkv", eps=eps))
            right = dict(kind="gated_delta", position=None, out=None, params=dict(
                name="mix.right", hidden=h, heads=r["heads"], kv_heads=r["kv_heads"], dim=r["dim"], vdim=r["vdim"],
                conv=r["conv"], eps=eps))
            mixer = PartSpec("side_by_side", dict(name="mix", hidden=h, eps=eps, combine="weighted",
                                                  scales=[m["left_scale"], m["right_scale"]], branches=[left, right]))
        elif layer.type == "lightning":
            mixer = PartSpec("retention", dict(name="mix", hidden=h, heads=m["heads"], dim=m["dim"], vdim=m["vdim"],
                                               decay=list(m["decay"]), rot_dims=0, activation="silu", k_scale=1.0, norm="row",
                                               gate="sigmoid", eps=eps))
        else:
            raise ConfigError(f"layer {i}: unknown mixer type '{layer.type}'")
        parts = dict(mixer_norm=norm("norm1"), mixer=mixer)
        if layer.mlp is not None:
            parts.update(feed_forward_norm=norm("norm2"), feed_forward=PartSpec("clamped_glu", dict(
                name="mlp", hidden=h, intermediate=layer.mlp["ff"], limit=layer.mlp["limit"], alpha=GLU_ALPHA,
                shift=GLU_SHIFT, bias=False)))
        layers.append(LayerSpec(prefix=f"l{i}", arrangement="prenorm", parts=parts, position=None))
    n = len(layers)
    schedule = [Run(i) for i in range(n)]
    if cfg.loop_times:
        entry = n                    # the junction ahead of every pass is one more "layer" of the spec
        layers.append(LayerSpec(prefix="loop", arrangement="junction", parts=dict(junction=PartSpec("loop_step", dict(
            hidden=h, passes=cfg.loop_times, step_name="loop.step")))))
        schedule = [Run(i) for i in range(cfg.loop_start)]
        for t in range(cfg.loop_times):
            schedule.append(Run(entry, params={"pass": t}))
            schedule += [Run(i, params={"pass": t}) for i in range(cfg.loop_start, cfg.loop_stop)]
        schedule += [Run(i) for i in range(cfg.loop_stop, n)]
    return ModelSpec(
        architecture=ZetivikConfig.ARCHITECTURE, hidden_size=h, vocab_size=cfg.vocab, max_position=MAX_POSITION,
        embedding=PartSpec("token_embedding", dict(vocab=cfg.vocab, hidden=h, weight_name="embed")),
        final_norm=PartSpec("group_rmsnorm", dict(weight_name="final.norm", hidden=h, eps=eps, groups=1, weight_offset=1.0)),
        lm_head=PartSpec("linear_head", dict(weight_name="head", vocab=cfg.vocab, hidden=h, tied_to="embed",
                                             softcap=cfg.logit_softcap)),
        positions=positions, layers=layers, schedule=schedule)


register_architecture(ZetivikConfig.ARCHITECTURE, ZetivikConfig, build_zetivik_spec, model_type=ZetivikConfig.MODEL_TYPE)
