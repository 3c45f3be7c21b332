"""The Kibilix architecture restated from its equations: float64, no paging, no slots, no kernels, one function
per mechanism.  It shares no code with the engine; the tests hold the engine against it.

Notation: ``X`` the streams ``[T, S, D]``, weights ``[out, in]`` applied as ``W v``, positions from 0.  Functions that
carry something from one portion of a sequence to the next take and return it (``state``), so the tests can also
cut a sequence and hand it over.  ``w`` is the dictionary of a model's tensors by name (float64).
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
#: None, or a type to which every matrix product's input and result, what is cached and what is activated are
#: rounded: that run is the model of what rounding alone does to the logits.
ROUND = [None]


def _r(v):
    return v if ROUND[0] is None else v.to(ROUND[0]).to(F64)


def silu(v):
    return v * torch.sigmoid(v)


def rms(v, eps):
    """The last dimension divided by its root mean square."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def linear(v, w, name):
    return _r(_r(v) @ w[name].T)


# ---------------------------------------------------------------------------------------------- embedding
def bigram_rows(tokens, buckets, mul_prev, mul_cur, previous=None):
    """Which row of the bigram table every token adds: the hash of the token before it and itself, or the row behind
    the hashed ones where there is no token before."""
    rows = []
    for t in tokens:
        rows.append(buckets if previous is None else (int(previous) * mul_prev + int(t) * mul_cur) % buckets)
        previous = t
    return torch.tensor(rows)


def embedding(cfg, w, tokens, previous=None):
    x = w["embed"][torch.as_tensor(tokens)]
    b = (cfg.get("embedding") or {}).get("bigram")
    if b:
        x = x + w["bigram"][bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"], previous)]
    return x


# ---------------------------------------------------------------------------------------------- streams
def read_streams(X, weights):
    """u = sum_s weights[s] X_s."""
    return torch.einsum("tsd,s->td", X, weights)


def join_streams(X, mix, out, y, factor):
    """X_t <- sum_s mix[s, t] X_s + factor * out[t] * y."""
    return torch.einsum("tsd,sr->trd", X, mix) + factor * out[None, :, None] * y[:, None, :]


# ---------------------------------------------------------------------------------------------- attention
def frequencies(dims, base, scaling=None):
    """base^(-2i/dims), where ``scaling`` is given stretched by ``factor`` for wavelengths beyond original / low, kept for
    those short of original / high, blended between."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > original / low:
                f = f / factor
            elif not wave < original / high:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_halves(x, positions, dims, base, scaling=None):
    """x ``[T, heads, dim]``: of the first ``dims`` dimensions, (i, i + dims/2) turn by position * f_i."""
    half = dims // 2
    a = (positions.to(F64)[:, None] * frequencies(dims, base, scaling)[None, :])[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., dims:]], dim=-1)


def chunk_visible(positions, size):
    """[T, T]: whether the query in row i sees the key in column j: not later, and in the same stretch of ``size``
    positions counted from 0 (every earlier key without a size)."""
    past = positions[:, None] >= positions[None, :]
    if not size:
        return past
    return past & ((positions[:, None] // size) == (positions[None, :] // size))


def capped(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def attention(h, w, name, m, positions=None):
    """Grouped-query attention inside chunks, scores capped, heads partly rotated."""
    t = h.shape[0]
    nh, d = m["heads"], m["dim"]
    nkv, vd, scale = m.get("kv_heads") or nh, m.get("vdim") or d, m.get("scale") or d ** -0.5
    pos = torch.arange(t) if positions is None else positions
    q, k = linear(h, w, name + ".q").reshape(t, nh, d), linear(h, w, name + ".k").reshape(t, nkv, d)
    rot = m.get("rot") or {}
    if rot.get("dims"):
        q, k = (rotate_halves(x, pos, rot["dims"], rot["base"], rot.get("scaling")) for x in (q, k))
    q, k, v = _r(q), _r(k), linear(h, w, name + ".v").reshape(t, nkv, vd)
    seen = chunk_visible(pos, (m.get("mask") or {}).get("size"))
    out = torch.zeros((t, nh, vd), dtype=F64)
    for head in range(nh):
        kv = head // (nh // nkv)
        s = capped((q[:, head] @ k[:, kv].T) * scale, m.get("softcap")).masked_fill(~seen, -math.inf)
        out[:, head] = torch.softmax(s, dim=-1) @ v[:, kv]
    return linear(out.reshape(t, nh * vd), w, name + ".o")


# ---------------------------------------------------------------------------------------------- delta rule
def causal_convolution(u, taps, tail=None):
    """y_t[c] = sum_j taps[c, j] u_(t - n + 1 + j)[c] with zeros ahead of a sequence.  Returns (y, the last n - 1 rows)."""
    n = taps.shape[1]
    tail = torch.zeros((n - 1, u.shape[1]), dtype=F64) if tail is None else tail
    rows = torch.cat([tail, u])
    y = sum(rows[j:j + u.shape[0]] * taps[:, j] for j in range(n))
    return y, rows[rows.shape[0] - (n - 1):]


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_decay(h, w, name, heads, dim):
    """g = exp(-exp(A_log) softplus(W_a2 W_a1 h + dt_bias)), one a head and key channel: ``[T, heads, dim]``."""
    a = (linear(linear(h, w, name + ".a1"), w, name + ".a2") + w[name + ".dt_bias"]).reshape(-1, heads, dim)
    return torch.exp(-torch.exp(w[name + ".A_log"])[None, :, None] * torch.nn.functional.softplus(a, threshold=1e4))


def write_rate(h, w, name):
    return torch.sigmoid(linear(h, w, name + ".b"))


def delta_recurrence(q, k, v, g, beta, s):
    """Token by token and head by head S <- diag(g) S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q; the heads' q, k
    ``[T, heads, dim]``, v ``[T, heads, vdim]``, g ``[T, heads, dim]``, beta ``[T, heads]``.  Returns (o, S)."""
    o = torch.zeros_like(v)
    for i in range(q.shape[0]):
        s = g[i][:, :, None] * s
        u = beta[i][:, None] * (v[i] - torch.einsum("hdv,hd->hv", s, k[i]))
        s = s + k[i][:, :, None] * u[:, None, :]
        o[i] = torch.einsum("hdv,hd->hv", s, q[i])
    return o, s


def channel_delta(h, w, name, m, eps, state=None):
    """``state``: (S, the last rows of q, k and v ahead of their convolutions).  Returns (result, the state after the
    last token)."""
    t = h.shape[0]
    nh, d = m["heads"], m["dim"]
    nk, vd = m.get("kv_heads") or nh, m.get("vdim") or d
    s, tails = (torch.zeros((nh, d, vd), dtype=F64), [None] * 3) if state is None else (state[0].clone(), state[1])
    rows, new_tails = [], []
    for leaf, tail, shape in zip("qkv", tails, ((nk, d), (nk, d), (nh, vd))):
        y, tail = causal_convolution(linear(h, w, f"{name}.{leaf}"), w[f"{name}.{leaf}.conv"], tail)
        rows.append(_r(silu(y)).reshape(t, *shape))
        new_tails.append(tail)
    share = torch.arange(nh) // (nh // nk)
    q, k, v = unit(rows[0])[:, share] * d ** -0.5, unit(rows[1])[:, share], rows[2]
    o, s = delta_recurrence(q, k, v, channel_decay(h, w, name, nh, d), write_rate(h, w, name), s)
    gate = torch.sigmoid(linear(linear(h, w, name + ".g1"), w, name + ".g2")).reshape(t, nh, vd)
    o = rms(o, eps) * w[name + ".norm"] * gate
    return linear(o.reshape(t, nh * vd), w, name + ".o"), (s, new_tails)


# ---------------------------------------------------------------------------------------------- feed-forward
def squared_relu(h, w, name):
    return linear(torch.relu(linear(h, w, name + ".up")) ** 2, w, name + ".down")


def clamped_expert(h, w, name, limit):
    g = linear(h, w, name + ".gate").clamp(max=limit)
    u = linear(h, w, name + ".up").clamp(-limit, limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1.0), w, name + ".down")


def route(z, correction, top):
    """Scores s = softmax(z) over every router output; the ``top`` with the largest s + correction; their s over their
    sum (+ 1e-20).  Returns (chosen ``[T, top]``, weights)."""
    s = torch.softmax(z, dim=-1)
    chosen = torch.topk(s + correction, top, dim=-1).indices
    picked = torch.gather(s, 1, chosen)
    return chosen, picked / (picked.sum(-1, keepdim=True) + 1e-20)


def experts(h, w, name, m):
    """``experts`` gated feed-forwards and, behind them among the router's outputs, ``identity`` ones that return h."""
    n, top = m["router"]["experts"], m["router"]["top"]
    hr = _r(h)
    chosen, weights = route(hr @ w[name + ".router"].T, w[name + ".correction"], top)
    out = torch.zeros_like(h)
    for i in range(h.shape[0]):
        for e, f in zip(chosen[i].tolist(), weights[i]):
            out[i] += f * (hr[i] if e >= n else clamped_expert(hr[i:i + 1], w, f"{name}.e{e}", m["expert"]["limit"])[0])
    return out


def feed_forward(h, w, name, m):
    return experts(h, w, name, m) if m["kind"] == "moe" else squared_relu(h, w, name)


# ---------------------------------------------------------------------------------------------- the model
def schedule(cfg):
    """The layers in the order they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    return (list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"]
            + list(range(loop["stop"], n)))


def forward(cfg, w, tokens, collect=None):
    """Logits ``[T, vocab]`` of a whole sequence.  ``collect`` (a list) takes the sum of the streams after every layer run."""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    X = embedding(cfg, w, tokens)[:, None, :].repeat(1, cfg["streams"], 1)
    for layer in schedule(cfg):
        spec, name = cfg["layers"][layer], f"l{layer}"

        def sublayer(X, q, f):
            u = read_streams(X, w[f"{name}.hc{q}.in"])
            return join_streams(X, w[f"{name}.hc{q}.mix"], w[f"{name}.hc{q}.out"], f(rms(u, eps) * w[f"{name}.norm{q}"]), m)
        if spec["type"] == "attention":
            X = sublayer(X, 1, lambda h: attention(h, w, name + ".mix", spec["mixer"]))
        else:
            X = sublayer(X, 1, lambda h: channel_delta(h, w, name + ".mix", spec["mixer"], eps)[0])
        if spec.get("mlp"):
            X = sublayer(X, 2, lambda h: feed_forward(h, w, name + ".mlp", spec["mlp"]))
        if collect is not None:
            collect.append(X.sum(1))
    return _r(rms(X.sum(1), eps) * w["final.norm"]) @ w["head"].T
