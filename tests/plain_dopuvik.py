"""Dopuvik in float64 NumPy, one function per mechanism, token by token where that is the
plainest form.  It shares no code with the package: the tests compare the engine with it.

A model is a dict `cfg` (the nested config.json of the design) and a dict of float64 arrays
by tensor name.  `forward(cfg, w, tokens)` gives the logits of every position of one
sequence; `forward(..., layers_out=[])` also collects the stream as every layer leaves it.

    start:   x = scale * embed[token]
    layer:   x <- x + mixer(LN(x) * g1);  x <- x + moe(LN(x) * g2)
    output:  logit_scale * head . (LN(x) * g_final)

with LN(x) = (x - mean) / sqrt(mean((x - mean)^2) + eps).
"""
from __future__ import annotations

import math

import numpy as np


def layer_norm(x, eps):
    c = x - x.mean(axis=-1, keepdims=True)
    return c / np.sqrt((c ** 2).mean(axis=-1, keepdims=True) + eps)


def rms(x, eps):
    return x / np.sqrt((x ** 2).mean(axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.clip(z, -700.0, 700.0)))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def _sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


# ---- positions ------------------------------------------------------------------------------

def frequencies(rot):
    """(angle per position of each pair, factor on cosine and sine), YaRN-scaled if asked for."""
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


def rotate_halves(x, p, rot):
    """x [..., d] at position p: of the first rot.dims dimensions, i turns with i + dims/2."""
    if not rot:
        return x
    n = rot["dims"]
    f, m = frequencies(rot)
    c, s = np.cos(p * f) * m, np.sin(p * f) * m
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., n:]], axis=-1)


def rotate_pairs(x, p, rot):
    """x [..., d] at position p: of the first rot.dims dimensions, 2i turns with 2i + 1."""
    if not rot:
        return x
    n = rot["dims"]
    f, m = frequencies(rot)
    out = x.copy()
    for i in range(n // 2):
        c, s = math.cos(p * f[i]) * m, math.sin(p * f[i]) * m
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def visible(i, mask):
    """The positions that the query at i sees: its window, and before it the first tokens."""
    if not mask or not mask.get("size"):
        return list(range(i + 1))
    keep = mask.get("keep_first", 0)
    return [j for j in range(i + 1) if i - j < mask["size"] or j < keep]


# ---- mixers ---------------------------------------------------------------------------------

def grouped_attention(h, m, t):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (h @ t["q"].T + t["q.b"]).reshape(T, H, d)
    k = (h @ t["k"].T + t["k.b"]).reshape(T, G, d)
    v = (h @ t["v"].T + t["v.b"]).reshape(T, G, dv)
    rot = m.get("rot")
    q = np.stack([rotate_halves(q[p], p, rot) for p in range(T)])
    k = np.stack([rotate_halves(k[p], p, rot) for p in range(T)])
    out = np.zeros((T, H, dv))
    for i in range(T):
        see = visible(i, m.get("mask"))
        for hh in range(H):
            g = hh // (H // G)
            out[i, hh] = softmax(k[see, g] @ q[i, hh] * m["scale"]) @ v[see, g]
    return out.reshape(T, H * dv) @ t["o"].T + t["o.b"]


def latent_attention(h, m, t, eps):
    H, d, rd, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    cq = rms(h @ t["dq"].T, eps) * t["dq.norm"]
    q = (cq @ t["uq"].T).reshape(T, H, d + rd)
    down = h @ t["dkv"].T
    c = rms(down[:, :R], eps) * t["dkv.norm"]
    k = (c @ t["uk"].T).reshape(T, H, d)
    v = (c @ t["uv"].T).reshape(T, H, dv)
    rot = m.get("rot")
    qr = np.stack([rotate_pairs(q[p, :, d:], p, rot) for p in range(T)])
    kr = np.stack([rotate_pairs(down[p, R:], p, rot) for p in range(T)])
    out = np.zeros((T, H, dv))
    for i in range(T):
        see = visible(i, m.get("mask"))
        for hh in range(H):
            s = (k[see, hh] @ q[i, hh, :d] + kr[see] @ qr[i, hh]) * m["scale"]
            out[i, hh] = softmax(s) @ v[see, hh]
    return out.reshape(T, H * dv) @ t["o"].T


def causal_conv(x, filt, bias=None):
    """x [T, C], filt [C, taps] whose last column meets the current token, zeros before the start."""
    T, taps = x.shape[0], filt.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    out = sum(padded[j:j + T] * filt[:, j] for j in range(taps))
    return out if bias is None else out + bias


def delta_rule(q, k, v, g, beta, state=None):
    """Per head S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.  q, k [T, H, d],
    v [T, H, dv], g, beta [T, H].  Returns (o [T, H, dv], state [H, d, dv])."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2])) if state is None else state.copy()
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        for hh in range(H):
            S[hh] = g[i, hh] * S[hh]
            u = beta[i, hh] * (v[i, hh] - S[hh].T @ k[i, hh])
            S[hh] = S[hh] + np.outer(k[i, hh], u)
            out[i, hh] = S[hh].T @ q[i, hh]
    return out, S


def gated_delta(h, m, t, eps):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    act = {x: silu(causal_conv(h @ t[x].T, t[x + ".conv"])) for x in ("q", "k", "v")}
    unit = lambda x: x / np.sqrt((x ** 2).sum(axis=-1, keepdims=True) + 1e-6)
    q = unit(act["q"].reshape(T, G, d)) * d ** -0.5
    k = unit(act["k"].reshape(T, G, d))
    q, k = np.repeat(q, H // G, axis=1), np.repeat(k, H // G, axis=1)
    beta = sigmoid(h @ t["b"].T)
    g = np.exp(-np.exp(t["A_log"]) * softplus(h @ t["a"].T + t["dt_bias"]))
    o, _ = delta_rule(q, k, act["v"].reshape(T, H, dv), g, beta)
    y = rms(o, eps) * t["norm"] * silu(h @ t["g"].T).reshape(T, H, dv)
    return y.reshape(T, H * dv) @ t["o"].T


def parallel(h, m, t, eps):
    return m["left_scale"] * grouped_attention(h, m["left"], _sub(t, "left.")) + \
        m["right_scale"] * gated_delta(h, m["right"], _sub(t, "right."), eps)


def ssd_scan(x, B, C, dt, decay, D, state=None):
    """Per head S <- decay S + dt B x^T, y = S^T C + D x.  x [T, H, dv], B, C [T, H, N],
    dt, decay [T, H], D [H].  Returns (y [T, H, dv], state [H, N, dv])."""
    T, H, dv = x.shape
    S = np.zeros((H, B.shape[2], dv)) if state is None else state.copy()
    out = np.zeros((T, H, dv))
    for i in range(T):
        for hh in range(H):
            S[hh] = decay[i, hh] * S[hh] + dt[i, hh] * np.outer(B[i, hh], x[i, hh])
            out[i, hh] = S[hh].T @ C[i, hh] + D[hh] * x[i, hh]
    return out, S


def grouped_rms(y, groups, eps):
    """Every one of `groups` equal parts of a row by its own root mean square."""
    T, n = y.shape
    return rms(y.reshape(T, groups, n // groups), eps).reshape(T, n)


def mamba2(h, m, t, eps):
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, T = H * dv, h.shape[0]
    z, xbc, dt = np.split(h @ t["in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
    xbc = silu(causal_conv(xbc, t["conv"], t["conv.b"]))
    x, B, C = np.split(xbc, [inner, inner + G * N], axis=1)
    B = np.repeat(B.reshape(T, G, N), H // G, axis=1)
    C = np.repeat(C.reshape(T, G, N), H // G, axis=1)
    dt = softplus(dt + t["dt_bias"])
    y, _ = ssd_scan(x.reshape(T, H, dv), B, C, dt, np.exp(-np.exp(t["A_log"]) * dt), t["D"])
    y = y.reshape(T, inner) * silu(z)
    return (grouped_rms(y, m["norm_groups"], eps) * t["norm"]) @ t["o"].T


# ---- feed-forward ---------------------------------------------------------------------------

def choose(choice, top, groups=1, keep=1):
    """The `top` largest choice scores among the `keep` groups whose largest score is largest."""
    n = len(choice) // groups
    best = [max(choice[g * n:(g + 1) * n]) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: -best[g])[:keep]
    allowed = [e for e in range(len(choice)) if e // n in kept]
    return sorted(allowed, key=lambda e: -choice[e])[:top]


def moe(h, mlp, t):
    r = mlp["router"]
    grp = r.get("groups") or {"count": 1, "keep": 1}
    out = np.zeros_like(h)
    for i in range(h.shape[0]):
        s = softmax(t["router"] @ h[i])
        for e in choose(s + t["correction"], r["top"], grp["count"], grp["keep"]):
            if e >= r["experts"]:
                y = h[i]
            else:
                x = _sub(t, f"e{e}.")
                y = (silu(h[i] @ x["gate"].T) * (h[i] @ x["up"].T)) @ x["down"].T
            out[i] += s[e] * r["scale"] * y
    return out


# ---- the model ------------------------------------------------------------------------------

def layer(cfg, w, i, x):
    eps = cfg["norm"]["eps"]
    p = f"l{i}."
    L = cfg["layers"][i]
    h, t = layer_norm(x, eps) * w[p + "norm1"], _sub(w, p + "mix.")
    if L["type"] == "parallel":
        y = parallel(h, L["mixer"], t, eps)
    elif L["type"] == "mamba2":
        y = mamba2(h, L["mixer"], t, eps)
    elif L["type"] == "latent_attention":
        y = latent_attention(h, L["mixer"], t, eps)
    else:
        raise ValueError(L["type"])
    x = x + y
    if L.get("mlp") is not None:
        x = x + moe(layer_norm(x, eps) * w[p + "norm2"], L["mlp"], _sub(w, p + "mlp."))
    return x


def forward(cfg, w, tokens, layers_out=None):
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i in range(len(cfg["layers"])):
        x = layer(cfg, w, i, x)
        if layers_out is not None:
            layers_out.append(x.copy())
    return (layer_norm(x, eps) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"]
