"""A plain, slow statement of the Bekunex decoder in numpy float64, one function per mechanism,
for the tests to hold the engine against. It shares no code with the package: it reads a config
dict of the architecture's own keys and a dict of weight arrays by checkpoint name, and runs a
whole sequence at once, token after token where a mechanism is a recurrence (no cache, no
state carried between calls, latents expanded into keys and values).

Notation: n tokens, width d; a mixer's input is X [n, d]; H heads, r the latent's width.
"""
from __future__ import annotations

import math

import numpy as np


def same(x):
    return x


# ----------------------------------------------------------------------------- small pieces
def layer_norm(x, w, b, eps):
    """Mean taken off, divided by the root of the mean squared deviation + eps, then w and b."""
    dev = x - x.mean(axis=-1, keepdims=True)
    return dev / np.sqrt((dev * dev).mean(axis=-1, keepdims=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rotate_halves(x, positions, rot):
    """x [n, heads, size]: within the first rot['dims'] channels, channel i pairs with channel
    i + dims/2 and the pair turns by position * base^(-2i/dims); the rest pass."""
    if rot is None:
        return x
    dims, base = rot["dims"], float(rot["base"])
    half = dims // 2
    out = np.array(x, dtype=np.float64)
    for t, p in enumerate(positions):
        for i in range(half):
            a = p * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


# ----------------------------------------------------------------------------------- mixers
def softmax_attention(q, k, v, scale, window=None, sink=None):
    """q, k [n, H, a], v [n, H, b] -> [n, H, b]. Query i reads keys j with 0 <= i - j < window
    (None: every j <= i); exp(sink_h), unscaled and without a value, joins the denominator."""
    n, H, _ = q.shape
    out = np.zeros((n, H, v.shape[2]))
    for i in range(n):
        lo = 0 if window is None else max(0, i - window + 1)
        s = np.einsum("jha,ha->hj", k[lo:i + 1], q[i]) * scale
        m = s.max(axis=1)
        if sink is not None:
            m = np.maximum(m, sink)
        e = np.exp(s - m[:, None])
        den = e.sum(axis=1)
        if sink is not None:
            den = den + np.exp(sink - m)
        out[i] = np.einsum("hj,jhb->hb", e / den[:, None], v[lo:i + 1])
    return out


def latent_of(X, W, p, m, eps, rnd=same):
    """(c [n, r], rotated shared key part [n, rot_dim] or None) of a layer that makes its own."""
    r, width = m["kv_rank"], m.get("rot_dim", 0)
    both = rnd(X @ W[p + "dkv"].T)
    c = rnd(rms_norm(both[:, :r], W[p + "dkv.norm"], eps))
    if not width:
        return c, None
    turned = rotate_halves(both[:, None, r:], range(len(X)), m.get("rot"))[:, 0]
    return c, rnd(turned)


def latent_attention(X, W, p, m, eps, rnd=same, lent=None):
    """Attention whose keys and values are expanded from the latent c. A rotated part of every
    query meets one rotated key part that all heads share, where the mixer has it; a window
    (mask), a sink per head and a gate on the heads are there where the weights and the config
    say so. `lent` is the latent of another layer, for a mixer that has none of its own."""
    n, H, a, b = len(X), m["heads"], m["dim"], m["vdim"]
    width = m.get("rot_dim", 0)
    q = rnd(X @ W[p + "q"].T).reshape(n, H, a + width)
    c, shared = lent if lent is not None else latent_of(X, W, p, m, eps, rnd)
    k = (c @ W[p + "uk"].T).reshape(n, H, a)
    v = (c @ W[p + "uv"].T).reshape(n, H, b)
    if width:
        q = np.concatenate([q[:, :, :a], rnd(rotate_halves(q[:, :, a:], range(n), m.get("rot")))], axis=2)
        k = np.concatenate([k, np.repeat(shared[:, None, :], H, axis=1)], axis=2)
    window = (m.get("mask") or {}).get("size")
    o = softmax_attention(q, k, v, m["scale"], window, W.get(p + "sink")).reshape(n, H * b)
    if p + "g" in W:
        o = rnd(o) * sigmoid(rnd(X @ W[p + "g"].T))
    return rnd(o) @ W[p + "o"].T, (c, shared)


def causal_conv(x, w, bias):
    """x [n, c], w [c, taps]: y_t = bias + sum_j w[:, taps-1-j] x_(t-j), zeros before t = 0."""
    n, taps = len(x), w.shape[1]
    y = np.tile(np.asarray(bias, dtype=np.float64), (n, 1))
    for j in range(min(taps, n)):
        y[j:] += x[:n - j] * w[:, taps - 1 - j]
    return y


def channel_scan(x, dt, A, B, C, D):
    """x, dt [n, c], A [c, N], B, C [n, N], D [c]: S <- exp(dt A) S + (dt x) B^T with S [c, N],
    y = S C + D x."""
    S = np.zeros(A.shape)
    y = np.zeros(x.shape)
    for t in range(len(x)):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def selective_scan_mixer(X, W, p, m, rnd=same):
    inner, N, R = m["inner"], m["state"], m["dt_rank"]
    xz = rnd(X @ W[p + "in"].T)
    x = rnd(silu(causal_conv(xz[:, :inner], W[p + "conv"], W[p + "conv.b"])))
    dbc = rnd(x @ W[p + "x"].T)
    dt = softplus(dbc[:, :R] @ W[p + "dt"].T + W[p + "dt.b"])
    y = channel_scan(x, dt, -np.exp(W[p + "A_log"]), dbc[:, R:R + N], dbc[:, R + N:], W[p + "D"])
    return rnd(y * silu(xz[:, inner:])) @ W[p + "o"].T


# ------------------------------------------------------------------------------ feed-forward
def gated(X, W, p, rnd=same):
    return rnd(silu(rnd(X @ W[p + "gate"].T)) * rnd(X @ W[p + "up"].T)) @ W[p + "down"].T


def choose_experts(s, correction, top, groups, keep):
    """One token's scores s [E] -> the chosen experts. The choice goes by s + correction; the
    experts fall into `groups` runs of neighbours, a run counts as its two largest choice
    scores (or its only one), and all but the best `keep` runs are out (ties: the lower index)."""
    choice = s + correction
    runs = choice.reshape(groups, -1)
    strength = [sum(sorted(run, reverse=True)[:2]) for run in runs]
    best = sorted(range(groups), key=lambda g: (-strength[g], g))[:keep]
    size = runs.shape[1]
    open_to = [e for e in range(len(s)) if e // size in best]
    return sorted(open_to, key=lambda e: (-choice[e], e))[:top]


def choice_margin(s, correction, top, groups, keep):
    """How far the choice of one token is from another one: the smaller of the gap between the
    weakest open group and the strongest closed one and of the gap between the last expert
    chosen and the next (infinite where nothing is left out)."""
    choice = s + correction
    runs = choice.reshape(groups, -1)
    strength = np.sort([sum(sorted(run, reverse=True)[:2]) for run in runs])[::-1]
    gap = strength[keep - 1] - strength[keep] if keep < groups else math.inf
    best = sorted(range(groups), key=lambda g: -sum(sorted(runs[g], reverse=True)[:2]))[:keep]
    inside = np.sort(runs[best].ravel())[::-1]
    return min(gap, inside[top - 1] - inside[top] if len(inside) > top else math.inf)


def routed(X, W, p, mlp, rnd=same, margins=None):
    r = mlp["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    s = sigmoid(X @ W[p + "router"].T)
    out = np.zeros(X.shape)
    for t in range(len(X)):
        if margins is not None:
            margins[t] = min(margins[t], choice_margin(s[t], W[p + "correction"], r["top"], g["count"], g["keep"]))
        for e in choose_experts(s[t], W[p + "correction"], r["top"], g["count"], g["keep"]):
            out[t] += s[t, e] * r["scale"] * gated(X[t:t + 1], W, f"{p}e{e}.", rnd)[0]
    if mlp.get("shared"):
        out += gated(X, W, p + "shared.", rnd)
    return out


# ------------------------------------------------------------------------------------ model
def forward(cfg, W, tokens, layer_outputs=None, rnd=same, margins=None):
    """Logits [n, vocab] of a whole sequence. `layer_outputs`, a list, gets the stream after
    every layer; `margins`, a list, gets for every token the closest call of any of its routers.
    With `rnd` (a rounding to a 16-bit type) the sublayers' inputs, the
    projections' results and what the last products read are rounded, as a 16-bit engine
    stores them; the stream, the norms, the softmax, the router and the recurrence stay."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)].astype(np.float64)
    latents = {}
    if margins is not None:
        margins[:] = [math.inf] * len(x)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rnd(layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps))
        if layer["type"] == "mamba1":
            y = selective_scan_mixer(h, W, p + "mix.", m, rnd)
        else:
            lent = latents[m["kv_from"]] if m.get("kv_from") is not None else None
            y, latents[i] = latent_attention(h, W, p + "mix.", m, eps, rnd, lent)
        if layer.get("mlp") is not None:
            y = y + routed(h, W, p + "mlp.", layer["mlp"], rnd, margins)
        x = x + y
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    n = rnd(layer_norm(x, W["final.norm"], W["final.norm.b"], eps))
    return n @ W["head"].T * cfg.get("logit_scale", 1.0)


def greedy(cfg, W, prompt, n):
    """The n tokens that follow `prompt` when the largest logit is taken every time (ties: the
    lower id)."""
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(np.argmax(forward(cfg, W, seq)[-1]))
        out.append(tok)
        seq.append(tok)
    return out
