"""The Kibilix architecture against its plain restatement (plain_kibilix.py): every mechanism alone through its part
and kernels, then whole models of three tiny configurations that differ in every size, option and order of layers,
stepped whole, token by token, in portions down to two tokens, in mixed batches over a pool so small that pages and
state slots are used again, through bin/trace_run and through Engine.generate.  Weights are random; where random
weights would hide a fault the tests set keys and queries by hand so that one score stands out (the first key of a
chunk, the last one ahead of it, keys at page borders, the token itself), and slow the decays of single channels so
that a state lost far back would show."""
from __future__ import annotations

import copy
import random

import numpy as np
import pytest
import torch

import plain_kibilix as plain
from helpers import KB, TraceProcess, kibilix_tensors, make_kibilix_folder, random_tokens

DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
PTOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}
# Whole models.  float32: the largest difference as a fraction of the largest logit (5e-5, or three times what rounding
# the matrix products to float32 causes if that is more).  bfloat16: a position's root-mean-square error over the
# vocabulary as a fraction of the logits' root mean square, against three times what rounding alone causes there: the
# plain model run again with every matrix product's input and result and what is cached rounded to bfloat16.
MTOL = {torch.float32: 5e-5}
NAME = {torch.float32: "float32", torch.bfloat16: "bfloat16"}
gpu = pytest.mark.gpu


def _rel(got, want):
    got, want = torch.as_tensor(got).double().cpu(), torch.as_tensor(want).double().cpu()
    return float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))


def _row_err(got, want):
    got, want = torch.as_tensor(got).double().cpu(), torch.as_tensor(want).double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt())


def _for_dtype(cfg, dtype):
    """Which experts a token takes is a discrete choice: in bfloat16 the stream differs from the plain one by
    roundings that can turn a close call the other way, and the logits then differ entirely.  So bfloat16 whole
    models take every expert, identity ones included (the weights still vary with the token, the sort and the tiles
    are the same); the choice itself is tested in bfloat16 on the part alone, close calls left out, and in whole
    models in float32."""
    if dtype in (torch.float32, "float32"):
        return cfg
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer["mlp"] and layer["mlp"]["kind"] == "moe":
            r = layer["mlp"]["router"]
            r["top"] = r["experts"] + r.get("identity", 0)
    return cfg


def _plain_logits(cfg, w, toks, dtype):
    """(the plain logits, the limit for an engine of ``dtype`` against them)."""
    want = plain.forward(cfg, w, toks)
    single = dtype in (torch.float32, "float32")
    plain.ROUND[0] = torch.float32 if single else torch.bfloat16
    try:
        rounded = plain.forward(cfg, w, toks)
    finally:
        plain.ROUND[0] = None
    return want, max(MTOL[torch.float32], 3.0 * _rel(rounded, want)) if single else 3.0 * _row_err(rounded, want)


def _model_err(got, want, dtype):
    return _rel(got, want) if dtype in (torch.float32, "float32") else _row_err(got, want)


def _rand(shape, seed, scale=1.0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * scale


def _dense(y):
    from inferflux_b200.parts.base import PartialSums
    return y.tensor.sum(0) if isinstance(y, PartialSums) else y.float()


# ------------------------------------------------------------------ CPU: configuration, spec, cache plan, the plain code
def test_config_is_read_from_its_own_keys():
    from inferflux_b200.config import ConfigError, KibilixConfig, build_spec, load_config
    cfg = load_config(copy.deepcopy(KB["A"]))
    assert isinstance(cfg, KibilixConfig) and cfg.width == 64 and cfg.vocab_size == 300 and cfg.norm_eps == 1e-5
    assert cfg.streams == 3 and cfg.residual_mult == 0.8 and cfg.bigram == dict(buckets=101, mul_prev=53, mul_cur=11)
    assert [l.type for l in cfg.layers] == ["attention", "channel_delta", "attention"]
    assert (cfg.loop_start, cfg.loop_stop, cfg.loop_times) == (0, 2, 3)
    scaling = dict(factor=4.0, low=1.0, high=8.0, original=64.0)
    assert cfg.layers[0].mixer == dict(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.3, softcap=6.0, chunk=20,
                                       rot=dict(dims=12, base=1000.0, scaling=scaling))
    assert cfg.layers[1].mixer == dict(heads=4, kv_heads=2, dim=12, vdim=20, conv=4)
    assert cfg.layers[0].mlp == dict(kind="dense", ff=96) and cfg.layers[2].mlp is None
    assert cfg.layers[1].mlp == dict(kind="moe", ff=40, limit=1.0, experts=5, top=3, identity=2)
    bare = load_config(copy.deepcopy(KB["B"]))                             # absent keys: their defaults
    assert bare.bigram is None and bare.loop_times == 0 and bare.layers[1].mlp["identity"] == 0
    m = bare.layers[1].mixer
    assert (m["kv_heads"], m["scale"], m["rot"]["dims"], m["chunk"], m["softcap"]) == (3, 10 ** -0.5, 0, 7, None)
    assert bare.layers[3].mixer["chunk"] is None and bare.layers[0].mixer["kv_heads"] == 2
    for c in (cfg, bare, load_config(copy.deepcopy(KB["C"]))):
        assert load_config(c.to_dict()) == c
    spec = build_spec(cfg)
    assert sorted(spec.positions) == ["rot0", "rot1"] and [l.arrangement for l in spec.layers] == ["streams"] * 3
    assert [l.parts["mixer"].kind for l in spec.layers] == ["window_attention", "gated_delta", "window_attention"]
    assert [r.layer for r in spec.schedule] == [0, 1, 0, 1, 0, 1, 2]
    assert "feed_forward" not in spec.layers[2].parts and spec.lm_head.params["tied_to"] is None
    assert [r.layer for r in build_spec(load_config(dict(copy.deepcopy(KB["A"]), loop=dict(start=1, stop=3, times=1)))).schedule] == [0, 1, 2]
    assert [r.layer for r in build_spec(bare).schedule] == [0, 1, 2, 3]
    for breaker, text in [(lambda d: d["layers"][0].update(type="serial"), "type"), (lambda d: d.pop("width"), "width"),
                          (lambda d: d["layers"][0]["mixer"].pop("dim"), "dim"), (lambda d: d.update(streams=17), "streams"),
                          (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
                          (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(low=8.0), "scaling"),
                          (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
                          (lambda d: d["layers"][0]["mixer"].update(softcap=0.0), "softcap"),
                          (lambda d: d["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
                          (lambda d: d["layers"][1]["mixer"].pop("conv"), "conv"),
                          (lambda d: d["layers"][1]["mlp"]["router"].update(top=8), "top"),
                          (lambda d: d["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
                          (lambda d: d["layers"][1]["mlp"].update(kind="sparse"), "kind"),
                          (lambda d: d["embedding"]["bigram"].pop("buckets"), "buckets"),
                          (lambda d: d["embedding"]["bigram"].update(mul_prev=1 << 60), "64 bits"),
                          (lambda d: d["norm"].pop("eps"), "eps"), (lambda d: d["loop"].update(stop=4), "loop")]:
        bad = copy.deepcopy(KB["A"])
        breaker(bad)
        with pytest.raises(ConfigError, match=text):
            load_config(bad)


def test_cache_and_state_plan():
    from inferflux_b200.config import build_spec, load_config
    from inferflux_b200.engine import Model
    model = Model(build_spec(load_config(copy.deepcopy(KB["A"]))), torch.float32, "cpu")
    names = {w.name: tuple(w.shape) for w in model.weight_specs() if w.kind != "ignored"}
    assert names["embed"] == names["head"] == (300, 64) and names["bigram"] == (102, 64) and names["final.norm"] == (64,)
    assert names["l0.mix.q"] == (64, 64) and names["l0.mix.k"] == (32, 64) and names["l0.mix.v"] == (48, 64) and names["l0.mix.o"] == (64, 96)
    assert names["l0.hc1.in"] == names["l0.hc2.out"] == (3,) and names["l0.hc1.mix"] == (3, 3)
    assert names["l0.norm1"] == names["l0.norm2"] == (64,) and "l2.norm2" not in names and "l2.hc2.mix" not in names
    assert names["l1.mix.q"] == names["l1.mix.k"] == (24, 64) and names["l1.mix.v"] == (80, 64) and names["l1.mix.v.conv"] == (80, 4)
    assert names["l1.mix.a1"] == names["l1.mix.g1"] == (-1, 64) and names["l1.mix.a2"] == (48, -1) and names["l1.mix.g2"] == (80, -1)
    assert names["l1.mix.A_log"] == (4,) and names["l1.mix.dt_bias"] == (48,) and names["l1.mix.b"] == (4, 64) and names["l1.mix.norm"] == (20,)
    assert names["l1.mlp.router"] == (7, 64) and names["l1.mlp.correction"] == (7,) and names["l1.mlp.e4.gate"] == (40, 64)
    assert "l1.mlp.e5.gate" not in names and names["l0.mlp.up"] == (96, 64) and not any(n.endswith(".b") and ".mix.b" not in n for n in names)
    needs = [[(s.name, s.heads, s.width) for s in n.streams] + [n.window, n.chunk] for n in model.kv_needs]
    assert needs == [[("k", 2, 16), ("v", 2, 24), None, 20], [("k", 1, 32), ("v", 1, 32), None, 33]]
    assert model.runs_per_group == [3, 1]                                        # every pass of the loop has a cache of its own
    states = [{s.name: tuple(s.shape) for s in per_run} for per_run in model.state_needs]
    gd = {"gated_delta": (4, 12, 20), "gated_delta_tail": (3, 24 + 24 + 80)}
    assert states == [{}, gd, {}, gd, {}, gd, {}]
    assert [(s.name, s.shape, s.dtype) for s in model.slot_needs()[-1]] == [("last_token", (1,), torch.int32)]
    b = Model(build_spec(load_config(copy.deepcopy(KB["B"]))), torch.float32, "cpu")
    assert [(n.streams[0].width, n.chunk) for n in b.kv_needs] == [(10, 7), (6, None)]
    assert [s.name for s in b.state_needs[0]] == ["gated_delta"] and b.slot_needs()[-1] == []   # one tap reaches back nowhere


def test_plain_carry_over_and_closed_forms():
    """The plain implementation's own consistency: a sequence cut in two with state and tails handed over, the delta rule
    as a triangular system over the whole sequence, the streams' mix as a matrix, the frequency bands, the router."""
    cfg = KB["A"]
    _, t = kibilix_tensors(cfg, 3)
    w = {k: v.double() for k, v in t.items()}
    m, eps, name = cfg["layers"][1]["mixer"], cfg["norm"]["eps"], "l1.mix"
    h = _rand((11, 64), 1).double()
    whole, (s, _) = plain.channel_delta(h, w, name, m, eps)
    for cut in (1, 2, 4, 9):
        a1, s1 = plain.channel_delta(h[:cut], w, name, m, eps)
        a2, s2 = plain.channel_delta(h[cut:], w, name, m, eps, s1)
        assert torch.allclose(torch.cat([a1, a2]), whole) and torch.allclose(s2[0], s)
    # head 3 (which reads query and key head 1): u from one triangular solve over all eleven tokens
    act = lambda x: x * torch.sigmoid(x)
    conv = lambda leaf: act(plain.causal_convolution(h @ w[f"{name}.{leaf}"].T, w[f"{name}.{leaf}.conv"])[0])
    k, v = plain.unit(conv("k").reshape(11, 2, 12)[:, 1]), conv("v").reshape(11, 4, 20)[:, 3]
    g, beta = plain.channel_decay(h, w, name, 4, 12)[:, 3], plain.write_rate(h, w, name)[:, 3]
    assert float(g.min()) > 0 and float(g.max()) < 1 and float(g.std(1).min()) > 1e-3          # the channels do differ
    c = torch.cumsum(torch.log(g), 0)
    low = torch.tril(torch.einsum("id,jd,ijd->ij", k, k, torch.exp(c[:, None] - c[None])), -1) * beta[:, None]
    u = torch.linalg.solve_triangular(torch.eye(11, dtype=torch.float64) + low, beta[:, None] * v, upper=False)
    assert torch.allclose(s[3], (k * torch.exp(c[-1] - c)).T @ u)
    X, mix, y = _rand((5, 3, 4), 2).double(), _rand((3, 3), 3).double(), _rand((5, 4), 4).double()
    got = plain.join_streams(X, mix, torch.tensor([1.0, 0.0, 2.0], dtype=torch.float64), y, 0.5)
    assert torch.allclose(got[:, 1], sum(mix[s_, 1] * X[:, s_] for s_ in range(3)))
    assert torch.allclose(got[:, 2] - y, sum(mix[s_, 2] * X[:, s_] for s_ in range(3)))
    assert torch.allclose(plain.read_streams(X, torch.tensor([0.0, 1.0, -1.0], dtype=torch.float64)), X[:, 1] - X[:, 2])
    rows = plain.bigram_rows([5, 2, 2], 10, 7, 3)
    assert rows.tolist() == [10, (35 + 6) % 10, (14 + 6) % 10] and plain.bigram_rows([2], 10, 7, 3, previous=5).tolist() == [1]
    bands = plain.frequencies(12, 1000.0, dict(factor=4.0, low=1.0, high=8.0, original=64))
    f = [1000.0 ** (-2.0 * i / 12) for i in range(6)]
    assert bands[0] == f[0] and bands[5] == f[5] / 4 and all(f[i] / 4 <= bands[i] <= f[i] for i in range(6))
    assert any(f[i] / 4 * 1.01 < bands[i] < f[i] * 0.99 for i in range(6))                     # one lies between the bands
    z = torch.log(torch.tensor([[0.5, 0.3, 0.2]], dtype=torch.float64))
    ids, wts = plain.route(z, torch.tensor([0.0, 0.0, 0.15], dtype=torch.float64), 2)          # the correction chooses, the score weighs
    assert sorted(ids[0].tolist()) == [0, 2] and torch.allclose(wts.sort().values, torch.tensor([[0.2, 0.5]], dtype=torch.float64) / 0.7)
    assert plain.capped(torch.tensor(3.0), 2.0) == pytest.approx(2 * np.tanh(1.5)) and plain.capped(3.0, None) == 3.0
    seen = plain.chunk_visible(torch.arange(9), 4)
    assert seen.sum(1).tolist() == [1, 2, 3, 4, 1, 2, 3, 4, 1] and seen[5].nonzero().flatten().tolist() == [4, 5]
    assert plain.schedule(cfg) == [0, 1, 0, 1, 0, 1, 2] and plain.schedule(KB["B"]) == [0, 1, 2, 3]


# ------------------------------------------------------------------ GPU: the mechanisms alone
def _runner_for(cfg, dtype, seed, tokens=512, tensors=None, **kw):
    from inferflux_b200.config import EngineConfig
    from inferflux_b200.config.registry import build_spec
    from inferflux_b200.engine import Model, StepRunner
    config, made = kibilix_tensors(cfg, seed, **kw)
    tensors = tensors or made
    model = Model(build_spec(config), dtype, DEV)
    plain_w = {k: v.double() for k, v in tensors.items()}
    model.load({k: (v.to(dtype) if v.dim() > 1 and ".hc" not in k and not k.endswith(".conv") else v.float()).to(DEV)
                for k, v in tensors.items()})
    runner = StepRunner(model, EngineConfig(dtype=NAME[dtype], kv_cache_tokens=tokens, max_seqs=4))
    return model, runner, plain_w


def _mixer_in_portions(model, runner, x, portions, dtype, layer=0):
    """Call one layer's mixer alone on rows cut into portions of one request."""
    from inferflux_b200.engine import StepEntry
    info, block = model.runs[layer], model.blocks[layer]
    outs, pos = [], 0
    for n in portions:
        ctx = runner.build_context([StepEntry("r", [1] * n, [])])
        for table, part in model.positions.items():
            ctx.position_tables[table] = part.prepare(ctx)
        position = ctx.position_tables.get(block.position_name) if block.position_name else None
        outs.append(_dense(block.mixer.forward(x[pos:pos + n].to(dtype).to(DEV).contiguous(), ctx, info, position)))
        runner.kv.advance("r", n)
        pos += n
    runner.end("r")
    return torch.cat(outs)


def _one_layer(name, layer, **changes):
    cfg = dict(KB[name], layers=[copy.deepcopy(KB[name]["layers"][layer])], loop=None)
    cfg["layers"][0]["mixer"].update(changes)
    return cfg


def _mixer_cfg(kind, mixer, width):
    return dict(KB["A"], width=width, loop=None, layers=[dict(type=kind, mixer=mixer, mlp=None)])


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,streams", [(50, 2), (64, 3), (1000, 4), (64, 1), (37, 5), (24, 16), (2048, 4), (52, 7)])
def test_streams_mixed_and_read_by_the_norm(dtype, hidden, streams):
    """The copies mixed anew with a sublayer's result (a tensor, slices of it, float32 or bfloat16, none), read and normed
    in one kernel; with picked rows, where the copies stay; the plain sum of the last norm."""
    from inferflux_b200.parts.base import PartialSums
    from inferflux_b200.parts.junction import StreamJoin
    from inferflux_b200.parts.norm import StreamRMSNorm
    eps, tol, factor = 3e-6, (2e-6 if dtype == torch.float32 else 5e-3), 0.6
    part = StreamRMSNorm(dict(weight_name="norm1", reads="hc1.in", hidden=hidden, streams=streams, eps=eps), "l0", dtype, DEV)
    last = StreamRMSNorm(dict(weight_name="norm1", reads=None, hidden=hidden, streams=streams, eps=eps), "l0", dtype, DEV)
    join = StreamJoin(dict(name="hc1", streams=streams, factor=factor), "l0", dtype, DEV)
    w = {"l0.norm1": 1 + _rand((hidden,), 3, 0.3), "l0.hc1.in": _rand((streams,), 4), "l0.hc1.mix": _rand((streams, streams), 5),
         "l0.hc1.out": _rand((streams,), 6)}
    w64 = {k: v.double() for k, v in w.items()}
    on = lambda v: v.to(DEV)
    last.load({k: on(v) for k, v in w.items()})
    tensors = {k: on(v) for k, v in w.items()}
    part.load(tensors), join.load(tensors)
    X, y, ys = _rand((7, streams, hidden), 1, 3.0), _rand((7, hidden), 2), _rand((3, 7, hidden), 7)
    norm = lambda X, reads: plain.rms(plain.read_streams(X, reads), eps) * w64["l0.norm1"]
    got = part.forward(on(X), None)
    assert got.dtype == dtype and _rel(got, norm(X.double(), w64["l0.hc1.in"])) < tol
    half = y.to(torch.bfloat16)
    for value, plain_y in ((on(y), y.double()), (PartialSums(on(ys)), ys.double().sum(0)), (on(half), half.double())):
        stream = on(X.clone())
        want = plain.join_streams(X.double(), w64["l0.hc1.mix"], w64["l0.hc1.out"], plain_y, factor)
        got = part.forward(stream, join.pending(value, None, None))
        assert _rel(stream, want) < 1e-6 and _rel(got, norm(want, w64["l0.hc1.in"])) < tol
        stream, pick = on(X.clone()), torch.tensor([6, 0, 6], dtype=torch.int32, device=DEV)
        got = last.forward(stream, join.pending(value, None, None), rows=pick)
        assert torch.equal(stream.cpu(), X) and _rel(got, norm(want, torch.ones(streams).double())[[6, 0, 6]]) < tol
    if streams > 1:                                                  # from and to are not exchanged: that would show
        turned = plain.join_streams(X.double(), w64["l0.hc1.mix"].T, w64["l0.hc1.out"], plain_y, factor)
        assert _rel(turned, want) > 1e-2


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,streams,buckets,mp,mc", [(64, 3, 101, 53, 11), (50, 1, 7, 1, 0), (36, 2, 64, 99991, 31337), (64, 4, 1, 5, 3)])
def test_token_pairs_across_portions_and_requests(dtype, hidden, streams, buckets, mp, mc):
    """The first token of a sequence, the first of a later portion (its predecessor waits in the slot), two requests in one
    step, and a slot taken again by a request that must not see the last one's token."""
    from inferflux_b200.engine import StepEntry
    cfg = dict(KB["A"], width=hidden, streams=streams, loop=None, layers=[copy.deepcopy(KB["A"]["layers"][0])],
               embedding=dict(bigram=dict(buckets=buckets, mul_prev=mp, mul_cur=mc)))
    model, runner, w = _runner_for(cfg, dtype, 11)
    a, b = random_tokens(300, 30, 1), random_tokens(300, 12, 2)
    a[7] = 0                                                         # token 0 as a predecessor is not "none"

    def run(entries):
        ctx = runner.build_context([StepEntry(r, t, []) for r, t in entries])
        out = model.embedding.forward_step(ctx)
        for r, t in entries:
            runner.kv.advance(r, len(t))
        assert tuple(out.shape[1:]) == (streams, hidden) and out.dtype == torch.float32
        assert all(torch.equal(out[:, s], out[:, 0]) for s in range(streams))
        return out[:, 0].cpu()

    want_a, want_b = plain.embedding(cfg, w, a), plain.embedding(cfg, w, b)
    got_a = [run([("a", a[:8])])]
    one = run([("b", b[:3]), ("a", a[8:9])])
    got_b, got_a = [one[:3]], got_a + [one[3:]]
    two = run([("a", a[9:11]), ("b", b[3:4])])
    got_a.append(two[:2]), got_b.append(two[2:])
    got_a.append(run([("a", a[11:])])), got_b.append(run([("b", b[4:])]))
    tol = 1e-6
    assert _rel(torch.cat(got_a), want_a) < tol and _rel(torch.cat(got_b), want_b) < tol
    if buckets > 1:
        assert _rel(plain.embedding(cfg, w, a, previous=a[0])[:1], want_a[:1]) > 1e-2      # what a first token takes does show
    runner.end("a"), runner.end("b")
    assert _rel(run([("c", b[:5])]), want_b[:5]) < tol and _rel(run([("d", a[:1])]), want_a[:1]) < tol
    runner.end("c"), runner.end("d")


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 0), ("A", 2), ("B", 1), ("B", 3), ("C", 1), ("C", 2)])
def test_attention_alone(dtype, name, layer):
    """Portions that start and end inside pages and chunks, single tokens across both, portions of two to seven tokens;
    grouped and ungrouped heads, whole, partial and no rotation, chunks shorter and longer than a page and none, caps and
    none; then the pages again."""
    cfg = _one_layer(name, layer)
    model, runner, w = _runner_for(cfg, dtype, 30 + layer, tokens=512)
    portions = [21, 1, 2, 1, 1, 10, 45, 1, 1, 2, 16, 1, 40, 7, 3]
    x = _rand((sum(portions), cfg["width"]), 31).to(dtype)
    m = cfg["layers"][0]["mixer"]
    want = plain.attention(x.double(), w, "l0.mix", m)
    got = _mixer_in_portions(model, runner, x, portions, dtype)
    assert _rel(got, want) < PTOL[dtype]
    again = _mixer_in_portions(model, runner, x[:9], [2, 7], dtype)
    assert _rel(again, want[:9]) < PTOL[dtype]
    runner.kv.check()
    for gone in ("softcap", "rot", "mask"):                          # every one of these shows in the result
        if gone in m:
            assert _rel(plain.attention(x.double(), w, "l0.mix", {k: v for k, v in m.items() if k != gone}), want) > 2e-2, gone
    if (m.get("rot") or {}).get("scaling"):
        other = dict(m, rot={k: v for k, v in m["rot"].items() if k != "scaling"})
        assert _rel(plain.attention(x.double(), w, "l0.mix", other), want) > 2e-2


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,vdim,width", [(16, 12, 64), (64, 64, 160), (128, 128, 320), (96, 96, 256)])
@pytest.mark.parametrize("chunk", [40, 48, 9])
def test_chunk_edges_with_one_score_that_stands_out(dtype, dim, vdim, width, chunk):
    """About 200 tokens, pages of 16.  Head 0's query is the token's first ``dim`` numbers and the key the next ``dim``; all
    tokens share one quiet key direction.  Each of the last eight tokens (around the last chunk's edge) gets a query that
    matches the key of one chosen token and no other: the first key of its chunk, the last one ahead of it, keys one before
    those, the very first token, the token just before, itself.  A visible target takes the weight, also under the cap; an
    edge that is off by one changes the result entirely.  The first queries come inside a portion, the others as single
    tokens."""
    edge = (200 // chunk) * chunk                                # the last chunk begins here
    n = edge + 5
    m = dict(heads=2, kv_heads=1, dim=dim, vdim=vdim, scale=14.0, softcap=20.0, mask=dict(size=chunk), rot=dict(dims=2, base=100.0))
    cfg = _mixer_cfg("attention", m, width)
    _, tensors = kibilix_tensors(cfg, 21, sharpen=1.0)
    eye = torch.eye(dim)
    tensors["l0.mix.q"] = torch.cat([torch.cat([eye, torch.zeros(dim, width - dim)], 1), _rand((dim, width), 22, 0.02)]).to(torch.bfloat16)
    tensors["l0.mix.k"] = torch.cat([torch.zeros(dim, dim), eye, torch.zeros(dim, width - 2 * dim)], 1).to(torch.bfloat16)
    model, runner, w = _runner_for(cfg, dtype, 21, tensors=tensors)
    x = _rand((n, width), 23, 0.3).to(torch.bfloat16).float()
    x[:, :2 * dim] = 0.0
    x[:, 2] = x[:, dim + 2] = 0.25                               # the shared direction (beyond the rotated pair)
    queries = list(range(edge - 3, n))
    prev = edge - chunk                                          # the chunk before the last begins here
    pairs = list(zip(queries, [prev, prev - 1, edge - 2, edge - 1, edge, 0, edge + 3, edge + 2],
                     [True, False, True, False, True, False, True, True]))
    for q, t, _ in pairs:
        u = torch.zeros(dim)
        u[3 + (q - queries[0])] = 1.0                            # a direction of its own for every pair
        if float(x[t, dim + 2]) == 0.25:
            x[t, dim:2 * dim] = 0.0
        x[t, dim:2 * dim] += u
        x[q, :dim] = u
    want = plain.attention(x.double(), w, "l0.mix", m)
    for q, t, visible in pairs:                                  # the plain result does rest on exactly the visible ones
        other = x.clone()
        other[t, dim:2 * dim] = 0.0
        other[t, dim + 2] = 0.25
        moved = plain.attention(other.double(), w, "l0.mix", m)[q]
        assert (_rel(moved, want[q]) > 0.1) == visible, (q, t)
    got = _mixer_in_portions(model, runner, x, [100, n - 100 - 6] + [1] * 6, dtype)
    assert _rel(got, want) < PTOL[dtype]
    short = _mixer_in_portions(model, runner, x, [n - 8, 2, 3, 2, 1], dtype)        # the same in short portions
    assert _rel(short, want) < PTOL[dtype]


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,kv_heads,chunk", [(64, 2, 700), (128, 1, None), (128, 4, 750), (40, 2, 700)])
def test_attention_over_a_long_context(dtype, dim, kv_heads, chunk):
    """A thousand tokens and chunks of hundreds, scores that reach well into the cap: single tokens whose keys the
    tensor-core kernel cuts into parts that a second kernel merges, right behind a chunk's edge and far from it."""
    m = dict(heads=4, kv_heads=kv_heads, dim=dim, scale=1.5 * dim ** -0.5, softcap=3.0, rot=dict(dims=dim, base=1e4))
    if chunk:
        m["mask"] = dict(size=chunk)
    cfg = _mixer_cfg("attention", m, 96)
    model, runner, w = _runner_for(cfg, dtype, 33, tokens=1024)
    portions = [600, 1, 1, 90, 1, 1, 4, 1, 1, 1, 1, 2, 45, 1, 1, 1, 240, 1, 1]
    x = _rand((sum(portions), 96), 34).to(dtype)
    want = plain.attention(x.double(), w, "l0.mix", m)
    assert _rel(plain.attention(x.double(), w, "l0.mix", dict(m, softcap=None)), want) > 0.05
    got = _mixer_in_portions(model, runner, x, portions, dtype)
    assert _rel(got, want) < PTOL[dtype]


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 1), ("B", 0), ("B", 2), ("C", 0), ("C", 3)])
def test_channel_delta_alone(dtype, name, layer):
    """Portions longer than several segments, portions of one and two tokens, single tokens (which move the convolutions'
    tails on in their own kernel); shared and unshared queries and keys, one tap to five, states of many shapes, inner
    sizes that are no multiple of anything; then the slot again, which the next request finds zeroed."""
    cfg = _one_layer(name, layer)
    model, runner, w = _runner_for(cfg, dtype, 40 + layer, tokens=512)
    portions = [150, 1, 1, 2, 64, 7, 1, 33, 16, 17]
    x = _rand((sum(portions), cfg["width"]), 41).to(dtype)
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    want, _ = plain.channel_delta(x.double(), w, "l0.mix", m, eps)
    got = _mixer_in_portions(model, runner, x, portions, dtype)
    assert _rel(got, want) < PTOL[dtype]
    again = _mixer_in_portions(model, runner, x[:10], [10], dtype)
    assert _rel(again, want[:10]) < PTOL[dtype]
    ones = _mixer_in_portions(model, runner, x[:40], [1] * 40, dtype)
    assert _rel(ones, want[:40]) < PTOL[dtype]
    flat = dict(w)                                               # one decay for all of a head's channels would show
    flat["l0.mix.a2"] = w["l0.mix.a2"].reshape(m["heads"], m["dim"], -1).mean(1, keepdim=True).repeat(1, m["dim"], 1).reshape(w["l0.mix.a2"].shape)
    assert _rel(plain.channel_delta(x.double(), flat, "l0.mix", m, eps)[0], want) > 2e-2


@gpu
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", [(2, 1, 128, 128, 4), (1, 1, 256, 40, 2), (3, 3, 7, 130, 16), (6, 2, 100, 33, 3), (2, 2, 1, 1, 4), (4, 2, 64, 64, 2), (8, 8, 128, 128, 4)])
def test_channel_delta_shapes(heads, kv_heads, dim, vdim, taps):
    """Heads from one number to the largest the kernels take, value sizes across their blocks' columns, few and many heads
    (narrow and wide column blocks)."""
    cfg = _mixer_cfg("channel_delta", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=taps), 48)
    model, runner, w = _runner_for(cfg, torch.float32, 43, tokens=512)
    portions = [70, 1, 1, 2, 31, 32, 33, 1]
    x = _rand((sum(portions), 48), 44)
    want, _ = plain.channel_delta(x.double(), w, "l0.mix", cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
    got = _mixer_in_portions(model, runner, x, portions, torch.float32)
    assert _rel(got, want) < PTOL[torch.float32]


@gpu
@pytest.mark.parametrize("case", ["kept", "gone", "alike", "frozen", "mixed"])
def test_channel_delta_at_its_ends(case):
    """``kept``: decays close to one and small rates, so that what the first token wrote still carries the result 300
    tokens on; ``gone``: decays of almost nothing, where only the token itself is left and running sums of logarithms
    reach thousands; ``alike``: every key the same, rates close to one, no decay, so that each token replaces the last
    one's value entirely (the triangular systems at their fullest); ``frozen``: rates of almost nothing, a state that
    never changes much; ``mixed``: in every head some channels forget at once and others keep everything."""
    cfg = _one_layer("A", 1)
    m, eps, name = cfg["layers"][0]["mixer"], cfg["norm"]["eps"], "l0.mix"
    _, t = kibilix_tensors(cfg, 5)
    a_log, dt, rate = {"kept": (-9.0, 0.0, -1.0), "gone": (3.0, 2.0, 0.0), "alike": (-20.0, 0.0, 9.0), "frozen": (-6.0, 0.0, -9.0),
                       "mixed": (0.0, 0.0, -1.0)}[case]
    x = _rand((300, 64), 6).to(torch.bfloat16).float()
    x[:, 0] = 1.0                                                    # a steady number for the rate to read
    t[f"{name}.A_log"], t[f"{name}.dt_bias"] = torch.full((4,), a_log).to(torch.bfloat16), torch.full((48,), dt).to(torch.bfloat16)
    if case == "mixed":
        t[f"{name}.a2"] = t[f"{name}.a2"] * 0
        t[f"{name}.dt_bias"] = torch.tensor([12.0, -14.0, 3.0] * 16).to(torch.bfloat16)
    t[f"{name}.b"] = t[f"{name}.b"] * 0
    t[f"{name}.b"][:, 0] = rate
    if case in ("kept", "mixed"):
        x[1:, 1:] *= 0.05
    if case == "alike":
        t[f"{name}.k"] = t[f"{name}.k"] * 0
        t[f"{name}.k"][:, 0] = 1.0
    model, runner, w = _runner_for(cfg, torch.float32, 5, tensors=t)
    want, _ = plain.channel_delta(x.double(), w, name, m, eps)
    g, beta = plain.channel_decay(x.double(), w, name, 4, 12), plain.write_rate(x.double(), w, name)
    if case in ("kept", "mixed"):
        lost, _ = plain.channel_delta(x.double()[1:], w, name, m, eps)
        assert _rel(lost[-1], want[-1]) > 0.02
    if case == "gone":
        assert float(torch.log(g).sum(0).max()) < -3000
    if case == "mixed":
        assert float(g.min()) < 1e-5 and float(g.max()) > 0.999999
    if case == "alike":
        assert float(beta.min()) > 0.999
    got = _mixer_in_portions(model, runner, x, [1, 2, 200, 90] + [1] * 7, torch.float32)
    assert _rel(got, want) < PTOL[torch.float32]


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ff,experts,identity,top,rows,limit", [
    (64, 40, 5, 2, 3, 7, 1.0), (50, 35, 3, 0, 2, 70, 0.5), (128, 64, 6, 3, 4, 300, 1.5), (64, 96, 4, 4, 8, 33, 30.0), (50, 18, 2, 1, 1, 1, 0.7),
    (72, 48, 40, 8, 5, 150, 1.0), (64, 64, 1, 3, 2, 300, 1.0)])
def test_experts_with_identity_and_a_corrected_choice(dtype, hidden, ff, experts, identity, top, rows, limit):
    """Few rows and many (short tiles and the tensor-core products), clamps that bite (and, at a limit of 30, never), more
    identity experts than others, every expert chosen; rows whose choice rests on a close call are left out."""
    from inferflux_b200.parts.feed_forward import RoutedExperts
    params = dict(name="mlp", hidden=hidden, intermediate=ff, experts=experts, identity=identity, top=top, activation="clamped_glu",
                  limit=limit, alpha=1.702, shift=1.0, route="all", correction=True, router_bias=False)
    part = RoutedExperts(params, "l0", dtype, DEV)
    scale = lambda n: 0.3 if "router" in n else 0.1 if "correction" in n else 0.3 if "down" not in n else 0.15
    w = {s.name: _rand(s.shape, 50 + i, scale(s.name)).to(torch.bfloat16).float() for i, s in enumerate(RoutedExperts.weight_specs(params, "l0"))}
    assert tuple(w["l0.mlp.router"].shape) == (experts + identity, hidden) and f"l0.mlp.e{experts}.up" not in w
    part.load({k: (v.to(dtype) if v.dim() > 1 else v).to(DEV) for k, v in w.items()})
    x = _rand((rows, hidden), 51, 1.0).to(dtype)
    w64 = {k: v.double() for k, v in w.items()}
    m = dict(router=dict(experts=experts, top=top), expert=dict(limit=limit))
    want = plain.experts(x.double(), w64, "l0.mlp", m)
    s = torch.softmax(x.double() @ w64["l0.mlp.router"].T, -1)
    ranked = torch.sort(s + w64["l0.mlp.correction"], dim=-1, descending=True)
    clear = torch.ones(rows, dtype=torch.bool)
    if top < experts + identity:
        clear = (ranked.values[:, top - 1] - ranked.values[:, top]) > 1e-4
        by_score = torch.sort(s, dim=-1, descending=True).indices[:, :top].sort(-1).values
        if rows > 30:
            assert bool((by_score != ranked.indices[:, :top].sort(-1).values).any())      # the correction does change choices
    if rows > 30 and identity:
        assert bool((ranked.indices[:, :top] >= experts).any())
    if rows > 30 and limit < 10:
        g = x.double() @ w64["l0.mlp.e0.gate"].T
        assert float((g > limit).double().mean()) > 0.02 and float((g < -limit).double().mean()) > 0.02
    assert int(clear.sum()) >= 0.8 * rows
    got = _dense(part.forward(x.to(DEV), None)).cpu()
    assert _rel(got[clear], want[clear]) < PTOL[dtype]


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ff,rows", [(64, 96, 3), (50, 35, 70), (128, 160, 300), (256, 1000, 8), (50, 45, 1), (128, 264, 200)])
def test_squared_relu_feed_forward(dtype, hidden, ff, rows):
    from inferflux_b200.parts.feed_forward import SquaredReluMLP
    params = dict(name="mlp", hidden=hidden, intermediate=ff)
    part = SquaredReluMLP(params, "l0", dtype, DEV)
    w = {s.name: _rand(s.shape, 60 + i, 0.15).to(torch.bfloat16).float() for i, s in enumerate(SquaredReluMLP.weight_specs(params, "l0"))}
    part.load({k: v.to(dtype).to(DEV) for k, v in w.items()})
    x = _rand((rows, hidden), 61).to(dtype)
    want = plain.squared_relu(x.double(), {k: v.double() for k, v in w.items()}, "l0.mlp")
    assert _rel(_dense(part.forward(x.to(DEV), None)), want) < PTOL[dtype]


# ------------------------------------------------------------------ GPU: whole models through the step function
def _logits_in_steps(runner, rid, toks, sizes):
    from inferflux_b200.engine import StepEntry
    outs, pos, k = [], 0, 0
    while pos < len(toks):
        n = min(sizes[k % len(sizes)], len(toks) - pos)
        outs.append(runner.step([StepEntry(rid, toks[pos:pos + n], list(range(n)))]).clone())
        pos, k = pos + n, k + 1
    runner.end(rid)
    return torch.cat(outs)


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_model_whole_one_by_one_and_in_portions(dtype, name):
    """The logits at every position for three ways of cutting the same prompt."""
    cfg = _for_dtype(KB[name], dtype)
    model, runner, w = _runner_for(cfg, dtype, ord(name), tokens=1024)
    toks = random_tokens(cfg["vocab"], 150, 31)
    want, limit = _plain_logits(cfg, w, toks, dtype)
    whole = _logits_in_steps(runner, "w", toks, [150])
    assert _model_err(whole, want, dtype) < limit
    ones = _logits_in_steps(runner, "o", toks[:90], [1])              # the captured decode graph after three steps
    assert runner.graph_replays > 0 and _model_err(ones, want[:90], dtype) < limit
    cut = _logits_in_steps(runner, "c", toks, [2, 3, 17, 1, 16, 5, 32, 2, 15, 64, 2])
    assert _model_err(cut, want, dtype) < limit
    if dtype == torch.float32:
        assert _rel(cut, whole) < 1e-5 and _rel(ones, whole[:90]) < 1e-5
    runner.kv.check(), runner.slots.check()


@gpu
def test_stream_after_every_layer():
    from inferflux_b200.engine import StepEntry
    cfg = KB["A"]
    model, runner, w = _runner_for(cfg, torch.float32, 9)
    toks = random_tokens(cfg["vocab"], 60, 4)
    want, seen = [], []
    plain.forward(cfg, w, toks, want)
    for block in model.blocks:
        def watched(residual, delta, ctx, run, inner=block.forward):
            out = inner(residual, delta, ctx, run)                    # what is pending is mixed in for the comparison
            mixed = torch.einsum("tsd,sr->trd", residual, out.mix) + out.out[None, :, None] * _dense(out.value)[:, None]
            seen.append(mixed.sum(1))
            return out
        block.forward = watched
    runner.step([StepEntry("s", toks, [0])])
    assert len(seen) == len(want) == 7 and all(_rel(g, x) < 2e-5 for g, x in zip(seen, want))


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_batches_of_unequal_requests_and_reused_slots(dtype, name):
    """Four requests of unequal length, portions beside single tokens, against each alone; then four more in
    the slots and pages the first ones gave back."""
    from inferflux_b200.engine import StepEntry
    cfg = _for_dtype(KB[name], dtype)
    model, runner, w = _runner_for(cfg, dtype, 41, tokens=4 * 128)
    rng = random.Random(3)
    for round_ in range(2):
        lens = [97, 5, 64, 33] if round_ == 0 else [31, 120, 2, 70]
        reqs = {f"r{round_}{i}": random_tokens(cfg["vocab"], n, 500 + 100 * round_ + 10 * i) for i, n in enumerate(lens)}
        want = {r: _plain_logits(cfg, w, t, dtype) for r, t in reqs.items()}
        alone = {}
        for r, t in reqs.items():                                  # each alone, its whole prompt in one step
            alone[r] = runner.step([StepEntry("alone", t, list(range(len(t))))]).clone()
            runner.end("alone")
        at, got = {r: 0 for r in reqs}, {r: [] for r in reqs}
        while any(at[r] < len(reqs[r]) for r in reqs):
            entries = []
            for r, t in reqs.items():
                left = len(t) - at[r]
                if left == 0 or (rng.random() < 0.2 and len(entries)):
                    continue
                n = 1 if left <= 6 else min(left - 6, rng.choice([1, 2, 3, 16, 29]))
                entries.append(StepEntry(r, t[at[r]:at[r] + n], list(range(n))))
            logits = runner.step(entries)
            row = 0
            for e in entries:
                got[e.rid].append(logits[row:row + len(e.tokens)].clone())
                row += len(e.tokens)
                at[e.rid] += len(e.tokens)
        for r in reqs:
            rows = torch.cat(got[r])
            ref, limit = want[r]
            assert _model_err(rows, ref, dtype) < limit, r
            assert _model_err(rows, alone[r], dtype) < (1e-5 if dtype == torch.float32 else limit), r
            runner.end(r)
        runner.kv.check(), runner.slots.check()
    assert all(p.reuses > 0 for p in runner.kv.pools)


@gpu
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_long_decoding_past_chunks(name):
    """300 tokens at once, then 200 one by one through the captured graph: chunks (of 7 to 48 tokens) begin and end
    among decoded tokens many times, their pages go back to the pool and come again, the states go on."""
    cfg = KB[name]
    model, runner, w = _runner_for(cfg, torch.float32, 51, tokens=512)
    toks = random_tokens(cfg["vocab"], 500, 52)
    want = plain.forward(cfg, w, toks)
    got = _logits_in_steps(runner, "d", toks, [300] + [1] * 200)
    assert runner.graph_replays >= 190 and _rel(got, want) < 5e-5
    chunked = [p for p, need in zip(runner.kv.pools, model.kv_needs) if need.chunk]
    assert chunked and all(p.reuses > 0 for p in chunked)


# ------------------------------------------------------------------ GPU: bin/trace_run and Engine.generate
@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_trace_replay_mixed_with_page_and_slot_reuse(name, dtype):
    """The command-line replay: the config.json picks the architecture; four state slots, a pool of the four
    longest requests; every request twice, so pages and slots turn over."""
    from helpers import load_plain_folder as load_plain
    cfg = _for_dtype(KB[name], dtype)
    folder = make_kibilix_folder(cfg, seed=60 + ord(name))
    pcfg, w = load_plain(folder)
    lengths = [70, 33, 5, 130, 64, 97, 1]
    requests = [random_tokens(cfg["vocab"], n, 1000 + 50 * i) for i, n in enumerate(lengths)]
    refs, limits = zip(*(_plain_logits(pcfg, w, r, dtype) for r in requests))
    # the rounding model's largest error over a handful of positions says little: short requests take the tightest limit
    # of the longer ones
    limits = [max(v, min(l for l, n in zip(limits, lengths) if n > 30)) for v in limits]
    pool = sum((n + 63) // 64 * 64 for n in sorted(lengths)[-4:])
    proc = TraceProcess(folder, dtype, pool)
    rng = random.Random(7)
    waiting = [(f"m{j}_{i}", i) for j, i in enumerate(list(range(len(requests))) * 2)]
    live, worst = {}, 0.0
    while waiting or live:
        while waiting and len(live) < 4:
            rid, i = waiting.pop(0)
            live[rid] = [i, 0]
        entries, ends, checks = [], [], []
        for rid, (i, pos) in list(live.items()):
            toks = requests[i]
            if rng.random() < 0.15 and len(live) > 1:
                continue
            left = len(toks) - pos
            n = 1 if left <= 20 else min(left - 20, rng.choice([2, 3, 7, 16, 29, 48]))
            want = list(range(n)) if n <= 3 else sorted(rng.sample(range(n), 3))
            entries.append(dict(id=rid, tokens=toks[pos:pos + n], want=want))
            checks.append((i, pos, want))
            live[rid][1] = pos + n
            if pos + n == len(toks):
                ends.append(rid)
                del live[rid]
        if not entries:
            continue
        got = proc.step(entries, end=ends)
        row = 0
        for i, pos, want in checks:
            for p in want:
                g = torch.tensor(got[row:row + 1].astype(np.float64))
                if dtype == "float32":
                    err = float((g[0] - refs[i][pos + p]).abs().max() / refs[i].abs().max())
                else:                                                  # the row's error on the whole request's scale
                    d = g[0] - refs[i][pos + p]
                    err = float((d - d.mean()).pow(2).mean().sqrt() / (refs[i] - refs[i].mean(-1, keepdim=True)).pow(2).mean().sqrt())
                worst = max(worst, err / limits[i])
                row += 1
    stats = proc.stats()
    assert proc.close() == 0
    assert worst < 1.0, worst
    assert all(u > 0 for u in stats["page_reuses"]) and stats["pages_free"] == stats["pages_total"]


@gpu
def test_greedy_generation_through_the_engine():
    """Engine.from_pretrained picks the architecture by config.json; the scheduler cuts prompts into portions of
    16 and batches them with decoding requests; float32 greedy continuations equal the plain ones."""
    from helpers import load_plain_folder as load_plain
    from inferflux_b200 import Engine, SamplingParams
    cfg = KB["A"]
    folder = make_kibilix_folder(cfg, seed=71)
    pcfg, w = load_plain(folder)
    prompts = [random_tokens(cfg["vocab"], n, 80 + n) for n in (5, 41, 17, 70, 3)]

    def plain_greedy(p, n):
        seq = list(p)
        for _ in range(n):
            seq.append(int(plain.forward(pcfg, w, seq)[-1].argmax()))
        return seq[len(p):]

    want = [plain_greedy(p, 12) for p in prompts]
    eng = Engine.from_pretrained(folder, dtype="float32", kv_cache_tokens=512, max_seqs=4, chunked_prefill_tokens=16)
    got = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    assert [g.tokens for g in got] == want
