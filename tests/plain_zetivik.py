"""The Zetivik architecture restated from its equations: float64, no paging, no slots, no kernels, one function
per mechanism.  It shares no code with the engine; the tests hold the engine against it.

Notation: ``x`` the stream ``[T, D]``, weights ``[out, in]`` applied as ``W v``, positions from 0.  Functions that
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


def zero_centred_norm(x, weight, eps):
    """RMS norm whose stored weight is the distance from one."""
    return rms(x, eps) * (1.0 + weight)


def linear(v, w, name):
    """``W v`` plus the bias ``<name>.b`` if ``w`` has it."""
    y = _r(v) @ w[name].T
    return _r(y + w[name + ".b"] if name + ".b" in w else y)


def rotate_halves(x, positions, dims, base):
    """x ``[T, heads, dim]``: of the first ``dims`` dimensions, (i, i + dims/2) turn by position * base^(-2i/dims)."""
    half = dims // 2
    f = base ** (-2.0 * torch.arange(half, dtype=F64) / max(dims, 1))
    a = (positions.to(F64)[:, None] * f[None, :])[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., dims:]], dim=-1)


def chunk_visible(positions, size):
    """[T, T]: whether the query in row i sees the key in column j: not later, and in the same stretch of ``size``
    positions counted from 0 (every earlier key without a size)."""
    past = positions[:, None] >= positions[None, :]
    if not size:
        return past
    return past & ((positions[:, None] // size) == (positions[None, :] // size))


def chunked_attention(h, w, name, m, eps, positions=None):
    """Grouped-query attention inside chunks; query and key heads normed with one weight of ``dim`` each, then
    rotated; one gate a head."""
    t = h.shape[0]
    nh, d = m["heads"], m["dim"]
    nkv, vd, scale = m.get("kv_heads") or nh, m.get("vdim") or d, m.get("scale") or d ** -0.5
    pos = torch.arange(t) if positions is None else positions
    q = rms(linear(h, w, name + ".q").reshape(t, nh, d), eps) * w[name + ".q.norm"]
    k = rms(linear(h, w, name + ".k").reshape(t, nkv, d), eps) * w[name + ".k.norm"]
    rot = m.get("rot") or {}
    if rot.get("dims"):
        q, k = rotate_halves(q, pos, rot["dims"], rot["base"]), rotate_halves(k, pos, rot["dims"], rot["base"])
    q, k, v = _r(q), _r(k), linear(h, w, name + ".v").reshape(t, nkv, vd)
    seen = chunk_visible(pos, (m.get("mask") or {}).get("size"))
    out = torch.zeros((t, nh, vd), dtype=F64)
    for head in range(nh):
        kv = head // (nh // nkv)
        s = ((q[:, head] @ k[:, kv].T) * scale).masked_fill(~seen, -math.inf)
        out[:, head] = torch.softmax(s, dim=-1) @ v[:, kv]
    out = out * torch.sigmoid(linear(h, w, name + ".g"))[:, :, None]
    return linear(out.reshape(t, nh * vd), w, name + ".o")


def causal_convolution(u, taps, tail=None):
    """y_t[c] = sum_j taps[c, j] u_(t - n + 1 + j)[c] with zeros ahead of a sequence.  Returns (y, the last n - 1 rows)."""
    n = taps.shape[1]
    tail = torch.zeros((n - 1, u.shape[1]), dtype=F64) if tail is None else tail
    rows = torch.cat([tail, u])
    y = sum(rows[j:j + u.shape[0]] * taps[:, j] for j in range(n))
    return y, rows[rows.shape[0] - (n - 1):]


def decay_and_rate(h, w, name):
    """g = exp(-exp(A_log) softplus(W_a h + dt_bias)) and beta = sigmoid(W_b h), one of each per head and token."""
    a = _r(h) @ w[name + ".a"].T + w[name + ".dt_bias"]
    g = torch.exp(-torch.exp(w[name + ".A_log"]) * torch.nn.functional.softplus(a, threshold=1e4))
    return g, torch.sigmoid(_r(h) @ w[name + ".b"].T)


def gated_delta(h, w, name, m, eps, state=None):
    """Per head S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q, token by token.  ``state``: (S, the last
    rows of q, k and v ahead of their convolutions).  Returns (result, the state after the last token)."""
    t = h.shape[0]
    nh, d = m["heads"], m["dim"]
    nk, vd = m.get("kv_heads") or nh, m.get("vdim") or d
    s, tails = (torch.zeros((nh, d, vd), dtype=F64), [None] * 3) if state is None else (state[0].clone(), state[1])
    rows, new_tails = [], []
    for leaf, tail, shape in zip("qkv", tails, ((nk, d), (nk, d), (nh, vd))):
        wt = {k: v for k, v in w.items() if k == f"{name}.{leaf}"}                  # '.b' beside these is no bias
        y, tail = causal_convolution(linear(h, wt, f"{name}.{leaf}"), w[f"{name}.{leaf}.conv"], tail)
        rows.append(_r(silu(y)).reshape(t, *shape))
        new_tails.append(tail)
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    q, k, v = unit(rows[0]) * d ** -0.5, unit(rows[1]), rows[2]
    g, beta = decay_and_rate(h, w, name)
    share = torch.arange(nh) // (nh // nk)
    o = torch.zeros((t, nh, vd), dtype=F64)
    for i in range(t):
        s = g[i][:, None, None] * s
        ki, qi = k[i][share], q[i][share]
        u = beta[i][:, None] * (v[i] - torch.einsum("hdv,hd->hv", s, ki))
        s = s + ki[:, :, None] * u[:, None, :]
        o[i] = torch.einsum("hdv,hd->hv", s, qi)
    o = rms(o, eps) * w[name + ".norm"] * silu(linear(h, w, name + ".g")).reshape(t, nh, vd)
    return linear(o.reshape(t, nh * vd), w, name + ".o"), (s, new_tails)


def parallel_mixer(h, w, name, m, eps, state=None):
    left = chunked_attention(h, w, name + ".left", m["left"], eps)
    right, state = gated_delta(h, w, name + ".right", m["right"], eps, state)
    return m.get("left_scale", 1.0) * left + m.get("right_scale", 1.0) * right, state


def lightning(h, w, name, m, eps, state=None):
    """S_t = decay_h S_(t-1) + k_t v_t^T and o_t = S_t^T q_t per head with silu'd q, k, v; all heads of a token
    normed together; a sigmoid gate.  Returns (result, the state after the last token)."""
    t = h.shape[0]
    nh, d = m["heads"], m["dim"]
    vd = m.get("vdim") or d
    q, k, v = (_r(silu(linear(h, w, f"{name}.{x}"))).reshape(t, nh, -1) for x in "qkv")
    s = torch.zeros((nh, d, vd), dtype=F64) if state is None else state.clone()
    decay = torch.tensor(m["decay"], dtype=F64)
    o = torch.zeros((t, nh, vd), dtype=F64)
    for i in range(t):
        s = decay[:, None, None] * s + k[i][:, :, None] * v[i][:, None, :]
        o[i] = torch.einsum("hdv,hd->hv", s, q[i])
    o = rms(o.reshape(t, nh * vd), eps) * w[name + ".norm"] * torch.sigmoid(linear(h, w, name + ".g"))
    return linear(o, w, name + ".o"), s


def clamped_glu(h, w, name, limit):
    g = linear(h, w, name + ".gate").clamp(max=limit)
    u = linear(h, w, name + ".up").clamp(-limit, limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1.0), w, name + ".down")


def schedule(cfg):
    """[(layer, number of the pass or None outside the loop)] in the order the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    return ([(i, None) for i in range(loop["start"])]
            + [(i, t) for t in range(loop["times"]) for i in range(loop["start"], loop["stop"])]
            + [(i, None) for i in range(loop["stop"], n)])


def forward(cfg, w, tokens, collect=None):
    """Logits ``[T, vocab]`` of a whole sequence.  ``collect`` (a list) takes the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens)]
    x = x0.clone()
    for layer, t in schedule(cfg):
        if t is not None and layer == cfg["loop"]["start"]:        # a pass begins
            x = (x if t == 0 else x + x0) + w["loop.step"][t]
        spec, name = cfg["layers"][layer], f"l{layer}"
        h = zero_centred_norm(x, w[name + ".norm1"], eps)
        mixer = {"parallel": parallel_mixer, "lightning": lightning}[spec["type"]]
        x = x + mixer(h, w, name + ".mix", spec["mixer"], eps)[0]
        if spec.get("mlp"):
            x = x + clamped_glu(zero_centred_norm(x, w[name + ".norm2"], eps), w, name + ".mlp", spec["mlp"]["limit"])
        if collect is not None:
            collect.append(x.clone())
    return softcap(_r(zero_centred_norm(x, w["final.norm"], eps)) @ w["embed"].T, cfg.get("logit_softcap"))


def softcap(logits, cap):
    return cap * torch.tanh(logits / cap) if cap else logits
