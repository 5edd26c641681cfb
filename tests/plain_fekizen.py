"""Fekizen in float64 NumPy, one function per mechanism, token by token where that is the
plainest form.  It shares no code with the package: the tests compare the engine with it.

A model is a dict `cfg` (the nested config.json of the design) and a dict of float64 arrays
by tensor name.  `forward(cfg, w, tokens)` gives the logits of every position of one
sequence; `forward(..., layers_out=[])` also collects the stream as every layer's run leaves it
(a layer of the repeated stretch once for every pass).

    start:   e = N(scale * embed[token] + pos[p]) * g_embed;  x = e
    layer:   h = N(x) * g1;  h_p <- h_p + (h_(p-1) - h_p) * shift  (h_(-1) = 0)
             x <- x + mixer(h);  x <- x + ff(N(x) * g2)
    repeat:  layers [start, stop) run `times` times; pass t begins with x <- x + step[t],
             every pass but the first with x <- x + e before that
    output:  head . (N(x) * g_final)

with N(x) = x / sqrt(mean(x^2) + eps).
"""
from __future__ import annotations

import math

import numpy as np


def rms(x, eps):
    return x / np.sqrt((x ** 2).mean(axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.clip(z, -700.0, 700.0)))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def token_shift(h, mix):
    """h [T, W]: every row moves towards the row before it, channel by channel."""
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mix


def yarn_frequencies(rot):
    """(angle per position of each pair, factor on cosine and sine)."""
    n, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def dim(turns):
        return n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim(s["fast"])), 0)
    hi = min(math.ceil(dim(s["slow"])), n - 1)
    out = []
    for i in range(n // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f[i] / s["factor"] * ramp + f[i] * (1.0 - ramp))
    return np.array(out), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, p, rot):
    """x [..., d] at position p: of the first rot.dims dimensions, i turns with i + dims/2 (no
    `rot`: nothing turns)."""
    if not rot:
        return x
    n = rot["dims"]
    f, m = yarn_frequencies(rot)
    c, s = np.cos(p * f) * m, np.sin(p * f) * m
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., n:]], axis=-1)


def seen_blocks(i, size, pool):
    """How many pooled blocks the query at position i sees: those whose last token is at most
    i - size."""
    b = 0
    while b * pool + pool - 1 <= i - size:
        b += 1
    return b


def attend(q, keys, values, scale, cap, sink):
    """One query over a list of keys and values; the denominator holds exp(sink) as well."""
    s = keys @ q * scale
    if cap:
        s = cap * np.tanh(s / cap)
    m = max(s.max(), sink)
    e = np.exp(s - m)
    return e @ values / (e.sum() + math.exp(sink - m))


def pooled_window_attention(h, m, t):
    """Grouped heads whose values are the unrotated keys; a window of single tokens, and older
    tokens as the mean keys and values of full blocks."""
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    size, P = m["mask"]["size"], m["mask"]["pool"]
    T = h.shape[0]
    q = (h @ t["q"].T).reshape(T, H, d)
    v = (h @ t["k"].T).reshape(T, G, d)
    k = np.stack([rotate(v[p], p, m.get("rot")) for p in range(T)])
    q = np.stack([rotate(q[p], p, m.get("rot")) for p in range(T)])
    full = T // P
    kb = k[:full * P].reshape(full, P, G, d).mean(axis=1)
    vb = v[:full * P].reshape(full, P, G, d).mean(axis=1)
    out = np.zeros((T, H, d))
    for i in range(T):
        lo, nb = max(0, i - size + 1), seen_blocks(i, size, P)
        for hh in range(H):
            g = hh // (H // G)
            keys = np.concatenate([kb[:nb, g], k[lo:i + 1, g]])
            vals = np.concatenate([vb[:nb, g], v[lo:i + 1, g]])
            out[i, hh] = attend(q[i, hh], keys, vals, m["scale"], m.get("softcap"), t["sink"][hh])
    return out.reshape(T, H * d) @ t["o"].T


def recurrence(q, k, v, decay, state=None):
    """Per head S <- diag(decay) S + k v^T, o = S^T q.  q, k [T, H, d], v [T, H, dv], decay
    [T, H, d].  Returns (o [T, H, dv], state [H, d, dv])."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2])) if state is None else state.copy()
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        for hh in range(H):
            S[hh] = decay[i, hh][:, None] * S[hh] + np.outer(k[i, hh], v[i, hh])
            out[i, hh] = S[hh].T @ q[i, hh]
    return out, S


def gated_linear_attention(h, m, t, eps, state=None):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (h @ t["q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ t["k"].T).reshape(T, H, d)
    v = (h @ t["v"].T).reshape(T, H, dv)
    z = (h @ t["a1"].T) @ t["a2"].T + t["a2.b"]
    decay = np.exp(log_sigmoid(z) / m["tau"]).reshape(T, H, d)
    o, S = recurrence(q, k, v, decay, state)
    y = (rms(o, eps) * t["norm"]).reshape(T, H * dv) * silu(h @ t["g"].T)
    return y @ t["o"].T, S


def lightning(h, m, t, eps, state=None):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = silu(h @ t["q"].T).reshape(T, H, d)
    k = silu(h @ t["k"].T).reshape(T, H, d)
    v = silu(h @ t["v"].T).reshape(T, H, dv)
    decay = np.broadcast_to(np.asarray(m["decay"], dtype=np.float64)[None, :, None], (T, H, d))
    o, S = recurrence(q, k, v, decay, state)
    y = rms(o.reshape(T, H * dv), eps) * t["norm"] * sigmoid(h @ t["g"].T)
    return y @ t["o"].T, S


def _sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def parallel_mixer(h, m, t, eps):
    left = pooled_window_attention(h, m["left"], _sub(t, "left."))
    right, _ = gated_linear_attention(h, m["right"], _sub(t, "right."), eps)
    return 0.5 * (rms(left, eps) * t["left.out"] + rms(right, eps) * t["right.out"])


def swiglu(h, t):
    return (silu(h @ t["gate"].T) * (h @ t["up"].T)) @ t["down"].T


def route(z, top):
    """Chosen experts of one token's router logits and the softmax over those logits alone."""
    chosen = np.argsort(-z, kind="stable")[:top]
    e = np.exp(z[chosen] - z[chosen].max())
    return chosen, e / e.sum()


def moe(h, mlp, t):
    out = np.zeros_like(h)
    for i in range(h.shape[0]):
        chosen, weights = route(t["router"] @ h[i], mlp["router"]["top"])
        for e, wgt in zip(chosen, weights):
            out[i] += wgt * swiglu(h[i], _sub(t, f"e{e}."))
    if mlp.get("shared"):
        out = out + swiglu(h, _sub(t, "shared."))
    return out


def layer(cfg, w, i, x):
    eps = cfg["norm"]["eps"]
    p = f"l{i}."
    L = cfg["layers"][i]
    h = token_shift(rms(x, eps) * w[p + "norm1"], w[p + "shift"])
    if L["type"] == "parallel":
        y = parallel_mixer(h, L["mixer"], _sub(w, p + "mix."), eps)
    elif L["type"] == "lightning":
        y, _ = lightning(h, L["mixer"], _sub(w, p + "mix."), eps)
    else:
        raise ValueError(L["type"])
    x = x + y
    if L.get("mlp") is not None:
        x = x + moe(rms(x, eps) * w[p + "norm2"], L["mlp"], _sub(w, p + "mlp."))
    return x


def run_order(cfg):
    """[(layer, pass or None: this call begins pass t of the repeated stretch)]"""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    order = [(i, None) for i in range(a)]
    for t in range(times):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def forward(cfg, w, tokens, layers_out=None):
    eps = cfg["norm"]["eps"]
    tokens = np.asarray(tokens)
    start = w["embed"][tokens] * cfg["embedding"]["scale"] + w["pos"][:len(tokens)]
    start = rms(start, eps) * w["embed.norm"]
    x = start
    for i, t in run_order(cfg):
        if t is not None:
            if t > 0:
                x = x + start
            x = x + w["loop.step"][t]
        x = layer(cfg, w, i, x)
        if layers_out is not None:
            layers_out.append(x.copy())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T
