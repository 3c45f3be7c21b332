"""``Kibilix`` as a spec: the one file that knows this architecture.

The embedding is a token's row plus a hashed row of the token pair, spread over several streams; every layer a
``streams`` block: a sublayer reads the RMS norm of a weighted sum of the streams, and its result joins all of them as
they are mixed anew.  Mixers: ``window_attention`` inside chunks (rotate-half positions, possibly scaled by wavelength
bands, capped scores) and ``gated_delta`` with one decay per head and key channel and a sigmoid gate, both projected in
two steps.  Feed-forwards: ``relu2_mlp``, ``routed_experts`` (clamped gated experts, identity experts, a correction of the
choice) or none.  A stretch of layers may run several times in a row on the same weights, every pass with caches and
states of its own.  The last norm reads the streams' sum.  Every distinct set of rotary parameters is one position
table, shared by the layers that use it.  Tensor names: ``embed``, ``bigram``, ``l<i>.{norm1,norm2}``,
``l<i>.{hc1,hc2}.{in,mix,out}``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import json

from ..config.model_config import KibilixConfig
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, Run

MAX_POSITION = 1 << 20      # the design has no longest sequence; this bounds the engine's bookkeeping
GLU_ALPHA, GLU_SHIFT = 1.702, 1.0       # an expert's two constants: g * sigmoid(1.702 g) * (u + 1)


def build_kibilix_spec(cfg: KibilixConfig) -> ModelSpec:
    h, eps, n_streams = cfg.width, cfg.norm_eps, cfg.streams
    positions, by_params = {}, {}

    def position_of(rot) -> str:
        """The name of the table for these rotary parameters (None if nothing rotates)."""
        if not rot["dims"]:
            return None
        key = json.dumps(rot, sort_keys=True)
        if key not in by_params:
            by_params[key] = f"rot{len(by_params)}"
            positions[by_params[key]] = PartSpec("rotary", dict(rotary_dim=rot["dims"], theta=rot["base"],
                                                                scaling=rot["scaling"]))
        return by_params[key]

    def norm(leaf, reads):
        return PartSpec("stream_rmsnorm", dict(weight_name=leaf, reads=reads, hidden=h, streams=n_streams, eps=eps))

    def join(name):
        return PartSpec("stream_join", dict(name=name, streams=n_streams, factor=cfg.residual_mult))
    layers = []
    for i, layer in enumerate(cfg.layers):
        m, position = layer.mixer, None
        if layer.type == "attention":
            position = position_of(m["rot"])
            mixer = PartSpec("window_attention", dict(
                name="mix", hidden=h, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], conv=0,
                rot_dims=m["rot"]["dims"], rot_layout="half", scale=m["scale"], softcap=m["softcap"], window=None,
                chunk=m["chunk"], sink=False, gate=None))
        else:
            mixer = PartSpec("gated_delta", dict(
                name="mix", hidden=h, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], conv=m["conv"],
                decay="channel", gate="sigmoid", two_step=True, eps=eps))
        parts = dict(mixer_norm=norm("norm1", "hc1.in"), mixer=mixer, mixer_join=join("hc1"))
        if layer.mlp is not None:
            f = layer.mlp
            if f["kind"] == "dense":
                ff = PartSpec("relu2_mlp", dict(name="mlp", hidden=h, intermediate=f["ff"]))
            else:
                ff = PartSpec("routed_experts", dict(
                    name="mlp", hidden=h, intermediate=f["ff"], experts=f["experts"], identity=f["identity"], top=f["top"],
                    activation="clamped_glu", limit=f["limit"], alpha=GLU_ALPHA, shift=GLU_SHIFT, route="all",
                    correction=True, router_bias=False))
            parts.update(feed_forward_norm=norm("norm2", "hc2.in"), feed_forward=ff, feed_forward_join=join("hc2"))
        layers.append(LayerSpec(prefix=f"l{i}", arrangement="streams", parts=parts, position=position))
    n = len(layers)
    order = list(range(n))
    if cfg.loop_times:
        order = (order[:cfg.loop_start] + order[cfg.loop_start:cfg.loop_stop] * cfg.loop_times + order[cfg.loop_stop:])
    return ModelSpec(
        architecture=KibilixConfig.ARCHITECTURE, hidden_size=h, vocab_size=cfg.vocab, max_position=MAX_POSITION,
        embedding=PartSpec("bigram_embedding", dict(vocab=cfg.vocab, hidden=h, table="embed", pairs="bigram", bigram=cfg.bigram,
                                                    streams=n_streams)),
        final_norm=PartSpec("stream_rmsnorm", dict(weight_name="final.norm", reads=None, hidden=h, streams=n_streams, eps=eps)),
        lm_head=PartSpec("linear_head", dict(weight_name="head", vocab=cfg.vocab, hidden=h, tied_to=None)),
        positions=positions, layers=layers, schedule=[Run(i) for i in order])


register_architecture(KibilixConfig.ARCHITECTURE, KibilixConfig, build_kibilix_spec, model_type=KibilixConfig.MODEL_TYPE)
