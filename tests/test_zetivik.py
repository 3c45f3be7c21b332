"""The Zetivik architecture against its plain restatement (plain_zetivik.py): every mechanism alone through its part
and kernels, then whole models of three tiny configurations that differ in every size, option and order of layers,
stepped whole, token by token, in portions down to two tokens, in mixed batches over a pool so small that pages and
state slots are used again, through bin/trace_run and through Engine.generate.  Weights are random; where random
weights would hide a fault the tests set keys and queries by hand so that one score stands out (the first key of a
chunk, the last one ahead of it, keys at page borders, the token itself), and slow the decays so that a state lost far
back would show."""
from __future__ import annotations

import copy
import random

import numpy as np
import pytest
import torch

import plain_zetivik as plain
from helpers import ZT, TraceProcess, make_zetivik_folder, random_tokens, zetivik_tensors

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
    from inferflux_b200.parts.base import PartialSums, ScaledSum
    if isinstance(y, ScaledSum):
        return sum(_dense(v) * f for v, f in y.terms)
    return y.tensor.sum(0) if isinstance(y, PartialSums) else y.float()


# ------------------------------------------------------------------ CPU: configuration, spec, cache plan, the plain code
def test_config_is_read_from_its_own_keys():
    from inferflux_b200.config import ConfigError, ZetivikConfig, build_spec, load_config
    cfg = load_config(copy.deepcopy(ZT["A"]))
    assert isinstance(cfg, ZetivikConfig) and cfg.width == 64 and cfg.vocab_size == 300 and cfg.norm_eps == 1e-5
    assert cfg.logit_softcap == 9.0 and [l.type for l in cfg.layers] == ["parallel", "lightning", "parallel"]
    assert (cfg.loop_start, cfg.loop_stop, cfg.loop_times) == (0, 2, 3)
    a = cfg.layers[0].mixer
    assert a["left"] == dict(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.3, chunk=20, rot=dict(dims=12, base=1000.0))
    assert a["right"] == dict(heads=4, kv_heads=2, dim=12, vdim=20, conv=4) and (a["left_scale"], a["right_scale"]) == (0.8, 1.3)
    assert cfg.layers[1].mixer == dict(heads=3, dim=12, vdim=20, decay=[0.999, 0.5, 0.9])
    assert cfg.layers[0].mlp == dict(kind="dense", ff=96, limit=2.0) and cfg.layers[1].mlp is None
    bare = load_config(copy.deepcopy(ZT["B"]))                             # absent keys: their defaults
    assert bare.logit_softcap is None and bare.loop_times == 0
    l, r = bare.layers[1].mixer["left"], bare.layers[1].mixer["right"]
    assert (l["kv_heads"], l["scale"], l["rot"]["dims"], l["chunk"]) == (3, 10 ** -0.5, 0, 7) and r["kv_heads"] == 2
    assert bare.layers[2].mixer["left"]["chunk"] is None and load_config(copy.deepcopy(ZT["C"])).layers[1].mixer["vdim"] == 64
    assert (bare.layers[1].mixer["left_scale"], bare.layers[1].mixer["right_scale"]) == (1.0, 1.0)
    assert load_config(cfg.to_dict()) == cfg and load_config(bare.to_dict()) == bare
    spec = build_spec(cfg)
    assert sorted(spec.positions) == ["rot0", "rot1"] and [l.arrangement for l in spec.layers] == ["prenorm"] * 3 + ["junction"]
    assert [l.parts["mixer"].kind for l in spec.layers[:3]] == ["side_by_side", "retention", "side_by_side"]
    assert [(r.layer, r.params.get("pass")) for r in spec.schedule] == [(3, 0), (0, 0), (1, 0), (3, 1), (0, 1), (1, 1), (3, 2), (0, 2), (1, 2), (2, None)]
    assert "feed_forward" not in spec.layers[1].parts and spec.lm_head.params["tied_to"] == "embed"
    once = build_spec(load_config(dict(copy.deepcopy(ZT["A"]), loop=dict(start=1, stop=3, times=1))))
    assert [r.layer for r in once.schedule] == [0, 3, 1, 2]                 # a single pass still gets its vector
    assert [r.layer for r in build_spec(bare).schedule] == [0, 1, 2]
    for breaker, text in [(lambda d: d["layers"][0].update(type="serial"), "type"), (lambda d: d.pop("width"), "width"),
                          (lambda d: d["layers"][0]["mixer"]["left"].pop("dim"), "dim"),
                          (lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "rot.dims"),
                          (lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
                          (lambda d: d["layers"][0]["mixer"]["right"].update(kv_heads=3), "kv_heads"),
                          (lambda d: d["layers"][0]["mixer"]["right"].pop("conv"), "conv"),
                          (lambda d: d["layers"][1]["mixer"].update(decay=[0.5, 0.5]), "decay"),
                          (lambda d: d["layers"][1]["mixer"].update(decay=[0.5, 0.5, 1.5]), "decay"),
                          (lambda d: d["norm"].pop("eps"), "eps"), (lambda d: d.update(logit_softcap=0.0), "softcap"),
                          (lambda d: d["loop"].update(stop=4), "loop"), (lambda d: d["layers"][0]["mlp"].pop("limit"), "limit"),
                          (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "kind")]:
        bad = copy.deepcopy(ZT["A"])
        breaker(bad)
        with pytest.raises(ConfigError, match=text):
            load_config(bad)


def test_cache_and_state_plan():
    from inferflux_b200.config import build_spec, load_config
    from inferflux_b200.engine import Model
    model = Model(build_spec(load_config(copy.deepcopy(ZT["A"]))), torch.float32, "cpu")
    names = {w.name: tuple(w.shape) for w in model.weight_specs() if w.kind != "ignored"}
    assert names["embed"] == (300, 64) and "head" not in names and names["final.norm"] == (64,) and names["loop.step"] == (3, 64)
    assert names["l0.mix.left.q"] == (64, 64) and names["l0.mix.left.k"] == (32, 64) and names["l0.mix.left.v"] == (48, 64)
    assert names["l0.mix.left.q.b"] == (64,) and names["l0.mix.left.v.b"] == (48,) and "l0.mix.left.o.b" not in names
    assert names["l0.mix.left.q.norm"] == names["l0.mix.left.k.norm"] == (16,) and names["l0.mix.left.g"] == (4, 64)
    assert names["l0.mix.left.o"] == (64, 96) and "l0.mix.left.out" not in names and "l0.mix.left.q.conv" not in names
    assert names["l0.mix.right.q"] == names["l0.mix.right.k"] == (24, 64) and names["l0.mix.right.v"] == (80, 64)
    assert names["l0.mix.right.q.conv"] == (24, 4) and names["l0.mix.right.v.conv"] == (80, 4)
    assert names["l0.mix.right.a"] == names["l0.mix.right.b"] == (4, 64) and names["l0.mix.right.norm"] == (20,)
    assert names["l0.mix.right.A_log"] == names["l0.mix.right.dt_bias"] == (4,) and names["l0.mix.right.g"] == (80, 64)
    assert names["l1.mix.q"] == (36, 64) and names["l1.mix.v"] == (60, 64) and names["l1.mix.norm"] == (60,)
    assert names["l0.mlp.gate"] == (96, 64) and "l0.mlp.gate.b" not in names and "l1.norm2" not in names
    needs = [[(s.name, s.heads, s.width) for s in n.streams] + [n.window, n.chunk] for n in model.kv_needs]
    assert needs == [[("k", 2, 16), ("v", 2, 24), None, 20], [("k", 1, 32), ("v", 1, 32), None, 33]]
    assert model.runs_per_group == [3, 1]                                        # every pass of the loop has a cache of its own
    states = [{s.name: tuple(s.shape) for s in per_run} for per_run in model.state_needs]
    gd, ln = {"gated_delta": (4, 12, 20), "gated_delta_tail": (3, 24 + 24 + 80)}, {"retention": (3, 12, 20)}
    assert states == [{}, gd, ln, {}, gd, ln, {}, gd, ln, {"gated_delta": (1, 16, 8), "gated_delta_tail": (2, 16 + 16 + 8)}]
    b = Model(build_spec(load_config(copy.deepcopy(ZT["B"]))), torch.float32, "cpu")
    assert [(n.streams[0].width, n.chunk) for n in b.kv_needs] == [(10, 7), (6, None)]
    assert [s.name for s in b.state_needs[1]] == ["gated_delta"]                 # one tap reaches back nowhere


@pytest.mark.parametrize("chunk,page", [(32, 16), (40, 16), (7, 16), (64, 64), (100, 8), (1, 4)])
def test_pages_of_a_chunk_that_is_over_go_back(chunk, page):
    """Whatever the step sizes, after every step exactly the pages that hold a position some later token sees, or
    that are not full, are held; a page that two chunks share stays until the later one is over."""
    from inferflux_b200.cache.kv_cache import KVCacheManager
    from inferflux_b200.parts.base import KVNeed
    need, plain_need = KVNeed.keys_and_values(1, 8, chunk=chunk), KVNeed.keys_and_values(1, 8)
    kv = KVCacheManager([need, plain_need], [80, 80], page)
    rng = random.Random(chunk)
    kv.add_request("a")
    n = 0
    while n < 300:
        step = min(rng.choice([1, 1, 2, 5, chunk, 37]), 300 - n)
        kv.reserve("a", step)
        for p in range(n, n + step):                          # what the step writes, and all that its tokens see
            assert kv.slot_of("a", 0, p) >= 0 and kv.slot_of("a", 0, p - p % chunk) >= 0
        kv.advance("a", step)
        n += step
        first = (n - n % chunk) // page                       # the next token's chunk begins in this block
        table = kv.block_table("a", 0)
        assert all(b < 0 for b in table[:first]) and all(b >= 0 for b in table[first:])
        assert all(b >= 0 for b in kv.block_table("a", 1))
        kv.check()
    kv.free_request("a")
    assert kv.num_free(0) == 80 and kv.num_free(1) == 80


def test_plain_carry_over_and_closed_forms():
    """The plain implementation's own consistency: sequences cut in two with state and tails handed over, the delta
    rule as a triangular system over the whole sequence, both recurrences as sums over earlier tokens, the chunks."""
    cfg = ZT["A"]
    _, t = zetivik_tensors(cfg, 3)
    w = {k: v.double() for k, v in t.items()}
    m, eps = cfg["layers"][0]["mixer"]["right"], cfg["norm"]["eps"]
    h = _rand((11, 64), 1).double()
    whole, (s, _) = plain.gated_delta(h, w, "l0.mix.right", m, eps)
    for cut in (1, 2, 4, 9):
        a1, s1 = plain.gated_delta(h[:cut], w, "l0.mix.right", m, eps)
        a2, s2 = plain.gated_delta(h[cut:], w, "l0.mix.right", m, eps, s1)
        assert torch.allclose(torch.cat([a1, a2]), whole) and torch.allclose(s2[0], s)
    # head 3 (which reads query and key head 1): u from one triangular solve over all eleven tokens
    name, act = "l0.mix.right", lambda x: x * torch.sigmoid(x)
    conv = lambda leaf: act(plain.causal_convolution(h @ w[f"{name}.{leaf}"].T, w[f"{name}.{leaf}.conv"])[0])
    k, v = conv("k").reshape(11, 2, 12)[:, 1], conv("v").reshape(11, 4, 20)[:, 3]
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    g, beta = plain.decay_and_rate(h, w, name)
    assert float(g.min()) > 0 and float(g.max()) < 1
    c = torch.cumsum(torch.log(g[:, 3]), 0)
    low = torch.tril(torch.exp(c[:, None] - c[None, :]) * (k @ k.T), -1) * beta[:, 3][:, None]
    u = torch.linalg.solve_triangular(torch.eye(11, dtype=torch.float64) + low, beta[:, 3][:, None] * v, upper=False)
    assert torch.allclose(s[3], (k * torch.exp(c[-1] - c)[:, None]).T @ u)
    lm = cfg["layers"][1]["mixer"]
    whole, s = plain.lightning(h, w, "l1.mix", lm, eps)
    a1, s1 = plain.lightning(h[:4], w, "l1.mix", lm, eps)
    a2, s2 = plain.lightning(h[4:], w, "l1.mix", lm, eps, s1)
    assert torch.allclose(torch.cat([a1, a2]), whole) and torch.allclose(s2, s)
    k, v = (act(h @ w[f"l1.mix.{x}"].T).reshape(11, 3, -1)[:, 2] for x in "kv")
    assert torch.allclose(s[2], sum(0.9 ** (10 - j) * torch.outer(k[j], v[j]) for j in range(11)))
    seen = plain.chunk_visible(torch.arange(9), 4)
    assert seen.sum(1).tolist() == [1, 2, 3, 4, 1, 2, 3, 4, 1] and seen[5].nonzero().flatten().tolist() == [4, 5]
    y = plain.causal_convolution(h, torch.tensor([[0.0, 1.0, 0.0]], dtype=torch.float64).repeat(64, 1))[0]
    assert torch.equal(y[1:], h[:-1]) and float(y[0].abs().max()) == 0.0         # the middle of three taps is the token before
    u, v = plain.rotate_halves(torch.eye(4, dtype=torch.float64).reshape(1, 4, 4), torch.tensor([2]), 2, 10.0)[0, :2]
    assert torch.allclose(u[:2], torch.tensor([np.cos(2.0), np.sin(2.0)])) and torch.allclose(v[:2], torch.tensor([-np.sin(2.0), np.cos(2.0)]))
    assert plain.schedule(cfg) == [(0, 0), (1, 0), (0, 1), (1, 1), (0, 2), (1, 2), (2, None)]
    assert plain.schedule(ZT["B"]) == [(0, None), (1, None), (2, None)]


# ------------------------------------------------------------------ GPU: the mechanisms alone
def _runner_for(cfg, dtype, seed, tokens=512, tensors=None, **kw):
    from inferflux_b200.config import EngineConfig
    from inferflux_b200.config.registry import build_spec
    from inferflux_b200.engine import Model, StepRunner
    config, made = zetivik_tensors(cfg, seed, **kw)
    tensors = tensors or made
    model = Model(build_spec(config), dtype, DEV)
    plain_w = {k: v.double() for k, v in tensors.items()}
    model.load({k: (v.to(dtype) if v.dim() > 1 else v.float()).to(DEV) for k, v in tensors.items()})
    runner = StepRunner(model, EngineConfig(dtype=NAME[dtype], kv_cache_tokens=tokens, max_seqs=4))
    return model, runner, plain_w


def _mixer_in_portions(model, runner, layer, x, portions, dtype, branch=None):
    """Call one layer's mixer (or one of its two branches) alone on rows cut into portions of one request."""
    from inferflux_b200.engine import StepEntry
    info, block = model.runs[layer], model.blocks[layer]
    mixer = block.mixer if branch is None else block.mixer.mixers[branch]
    outs, pos = [], 0
    for n in portions:
        ctx = runner.build_context([StepEntry("r", [1] * n, [])])
        for table, part in model.positions.items():
            ctx.position_tables[table] = part.prepare(ctx)
        name = block.mixer.branch_specs[branch]["position"] if branch is not None else None
        position = ctx.position_tables.get(name) if name else None
        outs.append(_dense(mixer.forward(x[pos:pos + n].to(dtype).to(DEV).contiguous(), ctx, info, position)))
        runner.kv.advance("r", n)
        pos += n
    runner.end("r")
    return torch.cat(outs)


def _one_layer(name, layer, **changes):
    cfg = dict(ZT[name], layers=[copy.deepcopy(ZT[name]["layers"][layer])], loop=None)
    cfg["layers"][0]["mixer"].update(changes)
    return cfg


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden", [50, 64, 1000])
def test_norm_around_zero_and_what_a_pass_adds(dtype, hidden):
    """The norm whose weight is stored as its distance from one: alone; with a weighted sum, rows and a vector that
    join it (each also absent) in one kernel; with picked rows behind pending sums."""
    from inferflux_b200.parts.base import JoinedSum, PartialSums, ScaledSum
    from inferflux_b200.parts.norm import GroupRMSNorm
    eps, tol = 3e-6, (2e-6 if dtype == torch.float32 else 5e-3)
    part = GroupRMSNorm(dict(weight_name="n", hidden=hidden, eps=eps, weight_offset=1.0), "", dtype, DEV)
    wt = _rand((hidden,), 3, 0.3).to(torch.bfloat16)
    part.load({"n": wt.to(DEV)})
    res, a, b, rows, vec = _rand((7, hidden), 1, 3.0), _rand((3, 7, hidden), 2), _rand((7, hidden), 4), _rand((7, hidden), 5), _rand((hidden,), 6)
    on = lambda v: v.to(DEV)
    norm = lambda x: plain.zero_centred_norm(x, wt.double(), eps)
    assert _rel(part.forward(on(res.clone()), None), norm(res.double())) < tol
    pair = ScaledSum([(PartialSums(on(a)), 0.7), (on(b), 1.9)])
    both = 0.7 * a.double().sum(0) + 1.9 * b.double()
    for value, add in ((pair, both), (PartialSums(on(a)), a.double().sum(0)), (on(b), b.double()), (None, 0.0)):
        for r, v in ((rows, vec), (None, vec), (rows, None)):
            stream = on(res.clone())
            want = res.double() + add + (r.double() if r is not None else 0) + (v.double() if v is not None else 0)
            got = part.forward(stream, JoinedSum(value, on(r) if r is not None else None, on(v) if v is not None else None))
            assert _rel(stream, want) < 1e-6 and _rel(got, norm(want)) < tol
    pick = torch.tensor([6, 0, 6], dtype=torch.int32, device=DEV)
    stream = on(res.clone())
    want = res.double() + both + rows.double() + vec.double()
    got = part.forward(stream, JoinedSum(pair, on(rows), on(vec)), rows=pick)
    assert _rel(stream, want) < 1e-6 and _rel(got, norm(want)[[6, 0, 6]]) < tol


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_capped_head_and_loop_step(dtype):
    from inferflux_b200.parts.base import RunInfo
    from inferflux_b200.parts.embedding import LinearHead
    from inferflux_b200.parts.junction import LoopStep
    table, x = _rand((77, 48), 1, 3.0).to(torch.bfloat16), _rand((5, 48), 2, 2.0).to(dtype)
    for cap in (4.0, 50.0, None):
        head = LinearHead(dict(vocab=77, hidden=48, weight_name="head", tied_to="embed", softcap=cap), "", dtype, DEV)
        head.load({"embed": table.to(dtype).to(DEV)})
        want = plain.softcap(x.double() @ table.double().T, cap)
        assert float(want.abs().max()) > 3.99 and _rel(head.forward(x.to(DEV)), want) < 2e-6 * (1 if dtype == torch.float32 else 10)
    step = LoopStep(dict(hidden=48, passes=3, step_name="loop.step"), "loop", dtype, DEV)
    step.load({"loop.step": _rand((3, 48), 3).to(DEV)})

    class Ctx:
        embedding_output = _rand((5, 48), 4).to(DEV)
    for t in range(3):
        got = step.pending(None, Ctx, RunInfo(0, params={"pass": t}))
        assert (got.rows is None) == (t == 0) and torch.equal(got.vector.cpu(), _rand((3, 48), 3)[t])


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ff,limit,rows", [(64, 96, 2.0, 3), (50, 35, 0.7, 70), (128, 160, 1.5, 300), (50, 45, 30.0, 1)])
def test_clamped_feed_forward_without_biases(dtype, hidden, ff, limit, rows):
    """Inputs large enough that both clamps bite (and, at a limit of 30, never), few rows and many."""
    from inferflux_b200.parts.feed_forward import ClampedGLU
    params = dict(name="mlp", hidden=hidden, intermediate=ff, limit=limit, bias=False)
    part = ClampedGLU(params, "l0", dtype, DEV)
    w = {s.name: _rand(s.shape, 50 + i, 0.3).to(torch.bfloat16).float() for i, s in enumerate(ClampedGLU.weight_specs(params, "l0"))}
    assert len(w) == 3
    part.load({k: v.to(dtype).to(DEV) for k, v in w.items()})
    x = _rand((rows, hidden), 51, 2.0).to(dtype)
    w64 = {k: v.double() for k, v in w.items()}
    want = plain.clamped_glu(x.double(), w64, "l0.mlp", limit)
    g = x.double() @ w64["l0.mlp.gate"].T
    assert (limit > 10) or (float((g > limit).double().mean()) > 0.02 and float((g < -limit).double().mean()) > 0.02)
    assert _rel(_dense(part.forward(x.to(DEV), None)), want) < PTOL[dtype]


def _attention_cfg(left, width):
    return dict(ZT["A"], width=width, loop=None, layers=[dict(type="parallel", mlp=None, mixer=dict(left=left, right=dict(heads=1, dim=4, vdim=4, conv=1)))])


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 0), ("A", 2), ("B", 1), ("B", 2), ("C", 0), ("C", 2)])
def test_chunked_attention_alone(dtype, name, layer):
    """The left branch: portions that start and end inside pages and chunks, single tokens across both, portions of two
    to seven tokens; grouped and ungrouped heads, whole, partial and no rotation, chunks shorter and longer than a page
    and none; then the pages again."""
    cfg = _one_layer(name, layer)
    model, runner, w = _runner_for(cfg, dtype, 30 + layer, tokens=512)
    portions = [21, 1, 2, 1, 1, 10, 45, 1, 1, 2, 16, 1, 40, 7, 3]
    x = _rand((sum(portions), cfg["width"]), 31).to(dtype)
    m, eps = cfg["layers"][0]["mixer"]["left"], cfg["norm"]["eps"]
    want = plain.chunked_attention(x.double(), w, "l0.mix.left", m, eps)
    got = _mixer_in_portions(model, runner, 0, x, portions, dtype, branch=0)
    assert _rel(got, want) < PTOL[dtype]
    again = _mixer_in_portions(model, runner, 0, x[:9], [2, 7], dtype, branch=0)
    assert _rel(again, want[:9]) < PTOL[dtype]
    runner.kv.check()
    for gone in ("q.b", "k.b", "v.b", "q.norm", "k.norm", "g"):                  # every one of these shows in the result
        other = dict(w)
        other[f"l0.mix.left.{gone}"] = torch.zeros_like(w[f"l0.mix.left.{gone}"]) + (1.0 if "norm" in gone else 0.0)
        assert _rel(plain.chunked_attention(x.double(), other, "l0.mix.left", m, eps), want) > 2e-2, gone


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,vdim,width", [(16, 12, 64), (64, 64, 160), (128, 128, 320), (96, 96, 256)])
@pytest.mark.parametrize("chunk", [40, 48, 9])
def test_chunk_edges_with_one_score_that_stands_out(dtype, dim, vdim, width, chunk):
    """205 tokens, pages of 16.  Head 0's query is the token's first ``dim`` numbers and the key the next ``dim``; all
    tokens share one quiet key and query direction.  Each of the last eight tokens (or the eight around the last
    chunk's edge) gets a query that matches the key of one chosen token and no other: the first key of its chunk, the
    last one ahead of it, keys one before those, the very first token, the token just before, itself.  A visible
    target takes the weight; an edge that is off by one changes the result entirely.  The first queries come inside a
    portion, the others as single tokens."""
    edge = (200 // chunk) * chunk                                # the last chunk begins here
    n = edge + 5
    left = dict(heads=2, kv_heads=1, dim=dim, vdim=vdim, scale=14.0 / dim, mask=dict(size=chunk), rot=dict(dims=2, base=100.0))
    cfg = _attention_cfg(left, width)
    _, tensors = zetivik_tensors(cfg, 21, sharpen=1.0)
    eye = torch.eye(dim)
    tensors["l0.mix.left.q"] = torch.cat([torch.cat([eye, torch.zeros(dim, width - dim)], 1), _rand((dim, width), 22, 0.05)]).to(torch.bfloat16)
    tensors["l0.mix.left.k"] = torch.cat([torch.zeros(dim, dim), eye, torch.zeros(dim, width - 2 * dim)], 1).to(torch.bfloat16)
    for leaf in ("q.b", "k.b"):
        tensors[f"l0.mix.left.{leaf}"] = torch.zeros_like(tensors[f"l0.mix.left.{leaf}"])
    for leaf in ("q.norm", "k.norm"):
        tensors[f"l0.mix.left.{leaf}"] = torch.ones_like(tensors[f"l0.mix.left.{leaf}"])
    model, runner, w = _runner_for(cfg, dtype, 21, tensors=tensors)
    x = _rand((n, width), 23, 0.3).to(torch.bfloat16).float()
    x[:, :2 * dim] = 0.0
    x[:, 2] = x[:, dim + 2] = 1.0                                # the shared direction (beyond the rotated pair)
    queries = list(range(edge - 3, n))
    prev = edge - chunk                                          # the chunk before the last begins here
    pairs = list(zip(queries, [prev, prev - 1, edge - 2, edge - 1, edge, 0, edge + 3, edge + 2],
                     [True, False, True, False, True, False, True, True]))
    for q, t, _ in pairs:
        u = torch.zeros(dim)
        u[3 + (q - queries[0])] = 1.0                            # a direction of its own for every pair
        if float(x[t, dim + 2]) == 1.0:
            x[t, dim:2 * dim] = 0.0
        x[t, dim:2 * dim] += u
        x[q, :dim] = u
    m, eps = left, cfg["norm"]["eps"]
    want = plain.chunked_attention(x.double(), w, "l0.mix.left", m, eps)
    for q, t, visible in pairs:                                  # the plain result does rest on exactly the visible ones
        other = x.clone()
        other[t, dim:2 * dim] = 0.0
        other[t, dim + 2] = 1.0
        moved = plain.chunked_attention(other.double(), w, "l0.mix.left", m, eps)[q]
        assert (_rel(moved, want[q]) > 0.1) == visible, (q, t)
    cut = [100, n - 100 - 6] + [1] * 6
    got = _mixer_in_portions(model, runner, 0, x, cut, dtype, branch=0)
    assert _rel(got, want) < PTOL[dtype]
    short = _mixer_in_portions(model, runner, 0, x, [n - 8, 2, 3, 2, 1], dtype, branch=0)        # the same in short portions
    assert _rel(short, want) < PTOL[dtype]


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,kv_heads,chunk", [(64, 2, 700), (128, 1, None), (128, 4, 750), (40, 2, 700)])
def test_chunked_attention_over_a_long_context(dtype, dim, kv_heads, chunk):
    """A thousand tokens and chunks of hundreds: single tokens whose keys the tensor-core kernel cuts into parts that a
    second kernel merges and gates, right behind a chunk's edge and far from it."""
    left = dict(heads=4, kv_heads=kv_heads, dim=dim, scale=0.5 * dim ** -0.5, rot=dict(dims=dim, base=1e4))
    if chunk:
        left["mask"] = dict(size=chunk)
    cfg = _attention_cfg(left, 96)
    model, runner, w = _runner_for(cfg, dtype, 33, tokens=1024)
    portions = [600, 1, 1, 90, 1, 1, 4, 1, 1, 1, 1, 2, 45, 1, 1, 1, 240, 1, 1]
    x = _rand((sum(portions), 96), 34).to(dtype)
    want = plain.chunked_attention(x.double(), w, "l0.mix.left", left, cfg["norm"]["eps"])
    got = _mixer_in_portions(model, runner, 0, x, portions, dtype, branch=0)
    assert _rel(got, want) < PTOL[dtype]


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 0), ("A", 2), ("B", 1), ("B", 2), ("C", 0), ("C", 2)])
def test_gated_delta_alone(dtype, name, layer):
    """The right branch: portions longer than several segments, portions of one and two tokens, single tokens (which
    move the convolutions' tails on in their own kernel); shared and unshared queries and keys, one tap to five, states
    of many shapes; then the slot again, which the next request finds zeroed."""
    cfg = _one_layer(name, layer)
    model, runner, w = _runner_for(cfg, dtype, 40 + layer, tokens=512)
    portions = [150, 1, 1, 2, 64, 7, 1, 33, 16, 17]
    x = _rand((sum(portions), cfg["width"]), 41).to(dtype)
    m, eps = cfg["layers"][0]["mixer"]["right"], cfg["norm"]["eps"]
    want, _ = plain.gated_delta(x.double(), w, "l0.mix.right", m, eps)
    got = _mixer_in_portions(model, runner, 0, x, portions, dtype, branch=1)
    assert _rel(got, want) < PTOL[dtype]
    again = _mixer_in_portions(model, runner, 0, x[:10], [10], dtype, branch=1)
    assert _rel(again, want[:10]) < PTOL[dtype]
    ones = _mixer_in_portions(model, runner, 0, x[:40], [1] * 40, dtype, branch=1)
    assert _rel(ones, want[:40]) < PTOL[dtype]


@gpu
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", [(2, 1, 128, 128, 4), (1, 1, 256, 40, 2), (3, 3, 7, 130, 16), (6, 2, 100, 33, 3), (2, 2, 1, 1, 4), (4, 2, 64, 64, 2)])
def test_gated_delta_shapes(heads, kv_heads, dim, vdim, taps):
    """Heads from one number to the largest the kernels take, value sizes across their blocks' columns."""
    cfg = dict(ZT["A"], width=48, loop=None, layers=[dict(type="parallel", mlp=None, mixer=dict(
        left=dict(heads=1, dim=4), right=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=taps)))])
    model, runner, w = _runner_for(cfg, torch.float32, 43, tokens=512)
    portions = [70, 1, 1, 2, 31, 32, 33, 1]
    x = _rand((sum(portions), 48), 44)
    want, _ = plain.gated_delta(x.double(), w, "l0.mix.right", cfg["layers"][0]["mixer"]["right"], cfg["norm"]["eps"])
    got = _mixer_in_portions(model, runner, 0, x, portions, torch.float32, branch=1)
    assert _rel(got, want) < PTOL[torch.float32]


@gpu
@pytest.mark.parametrize("case", ["kept", "gone", "alike", "frozen"])
def test_gated_delta_at_its_ends(case):
    """``kept``: decays close to one and small rates, so that what the first token wrote still carries the result 300
    tokens on; ``gone``: decays of almost nothing, where only the token itself is left and running sums of logarithms
    reach thousands; ``alike``: every key the same, rates close to one, no decay, so that each token replaces the last
    one's value entirely (the triangular systems at their fullest); ``frozen``: rates of almost nothing, a state that
    never changes much."""
    cfg = _one_layer("A", 0)
    m, eps = cfg["layers"][0]["mixer"]["right"], cfg["norm"]["eps"]
    _, t = zetivik_tensors(cfg, 5)
    a_log, dt, rate = {"kept": (-9.0, 0.0, -1.0), "gone": (3.0, 2.0, 0.0), "alike": (-20.0, 0.0, 9.0), "frozen": (-6.0, 0.0, -9.0)}[case]
    x = _rand((300, 64), 6).to(torch.bfloat16).float()
    x[:, 0] = 1.0                                                    # a steady number for the rate to read
    name = "l0.mix.right"
    t[f"{name}.A_log"], t[f"{name}.dt_bias"] = torch.full((4,), a_log).to(torch.bfloat16), torch.full((4,), dt).to(torch.bfloat16)
    t[f"{name}.b"] = t[f"{name}.b"] * 0
    t[f"{name}.b"][:, 0] = rate
    if case == "kept":
        x[1:, 1:] *= 0.05
    if case == "alike":
        t[f"{name}.k"] = t[f"{name}.k"] * 0
        t[f"{name}.k"][:, 0] = 1.0
    model, runner, w = _runner_for(cfg, torch.float32, 5, tensors=t)
    want, _ = plain.gated_delta(x.double(), w, name, m, eps)
    g, beta = plain.decay_and_rate(x.double(), w, name)
    if case == "kept":
        lost, _ = plain.gated_delta(x.double()[1:], w, name, m, eps)
        assert _rel(lost[-1], want[-1]) > 0.05
    if case == "gone":
        assert float(torch.log(g).sum(0).max()) < -3000
    if case == "alike":
        assert float(beta.min()) > 0.999
    got = _mixer_in_portions(model, runner, 0, x, [1, 2, 200, 90] + [1] * 7, torch.float32, branch=1)
    assert _rel(got, want) < PTOL[torch.float32]


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 1), ("B", 0), ("C", 1)])
def test_lightning_alone(dtype, name, layer):
    """Portions longer than several segments, of one and two tokens, single tokens; decays of one and of zero; then the
    slot again.  With a decay of 0.999 the first token's write still shows 300 tokens on."""
    cfg = _one_layer(name, layer)
    model, runner, w = _runner_for(cfg, dtype, 45 + layer, tokens=512)
    portions = [150, 1, 1, 2, 64, 7, 1, 33, 16, 17, 1, 1]
    x = _rand((sum(portions), cfg["width"]), 46).to(dtype)
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    want, _ = plain.lightning(x.double(), w, "l0.mix", m, eps)
    got = _mixer_in_portions(model, runner, 0, x, portions, dtype)
    assert _rel(got, want) < PTOL[dtype]
    again = _mixer_in_portions(model, runner, 0, x[:10], [10], dtype)
    assert _rel(again, want[:10]) < PTOL[dtype]
    if name != "C":
        y = x.double().clone()
        y[1:] *= 0.05
        far, _ = plain.lightning(y, w, "l0.mix", m, eps)
        lost, _ = plain.lightning(y[1:], w, "l0.mix", m, eps)
        assert _rel(lost[-1], far[-1]) > 0.02
        got = _mixer_in_portions(model, runner, 0, y.to(dtype), [1, 2, sum(portions) - 9] + [1] * 6, dtype)
        if dtype == torch.float32:
            assert _rel(got, far) < PTOL[dtype]


@gpu
@pytest.mark.parametrize("heads,dim,vdim", [(2, 128, 128), (1, 256, 20), (3, 7, 300), (2, 1, 1)])
def test_lightning_shapes(heads, dim, vdim):
    cfg = dict(ZT["A"], width=48, loop=None, layers=[dict(type="lightning", mlp=None, mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=[0.9, 1.0, 0.2][:heads]))])
    model, runner, w = _runner_for(cfg, torch.float32, 47, tokens=512)
    portions = [70, 1, 1, 2, 31, 32, 33, 1]
    x = _rand((sum(portions), 48), 48)
    want, _ = plain.lightning(x.double(), w, "l0.mix", cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
    got = _mixer_in_portions(model, runner, 0, x, portions, torch.float32)
    assert _rel(got, want) < PTOL[torch.float32]


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
    cfg = ZT[name]
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
    from inferflux_b200.parts.base import ScaledSum
    cfg = ZT["A"]
    model, runner, w = _runner_for(cfg, torch.float32, 9)
    toks = random_tokens(cfg["vocab"], 60, 4)
    want = []
    plain.forward(cfg, w, toks, want)
    seen = []
    for block in model.blocks:
        if not hasattr(block, "mixer"):
            continue                                                  # the junction ahead of a pass is no layer

        def watched(residual, delta, ctx, run, inner=block.forward):
            out = inner(residual, delta, ctx, run)
            seen.append(residual.clone() + (_dense(out) if out is not None else 0.0))    # pending sums included
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
    cfg = ZT[name]
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
    cfg = ZT[name]
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
    cfg = ZT[name]
    folder = make_zetivik_folder(cfg, seed=60 + ord(name))
    pcfg, w = load_plain(folder)
    lengths = [70, 33, 5, 130, 64, 97, 1]
    requests = [random_tokens(cfg["vocab"], n, 1000 + 50 * i) for i, n in enumerate(lengths)]
    refs, limits = zip(*(_plain_logits(pcfg, w, r, dtype) for r in requests))
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
    cfg = ZT["A"]
    folder = make_zetivik_folder(cfg, seed=71)
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
