"""A plain, slow statement of the Kesozen decoder in numpy float64, one function per mechanism, for
the tests to hold the engine against. It shares no code with the package: it reads a config dict of
the architecture's own keys and a dict of weight arrays by checkpoint name, and runs a whole
sequence at once, token after token where a mechanism is a recurrence (no cache, no state carried
between calls).

Notation: n tokens, width d; a mixer's input is X [n, d]; H query or value heads, G key heads.
"""
from __future__ import annotations

import math

import numpy as np


def same(x):
    return x


# ----------------------------------------------------------------------------- small pieces
def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


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


# --------------------------------------------------------------------------------- attention
def softmax_plus_one(q, k, v, scale):
    """q [n, H, a], k [n, G, a], v [n, G, b] -> [n, H, b]. Query i reads every key j <= i; the
    denominator has one more, as if a key with score 0 and no value stood beside them."""
    n, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((n, H, v.shape[2]))
    for h in range(H):
        s = scale * (q[:, h] @ k[:, h // per].T)
        s[np.triu_indices(n, 1)] = -np.inf
        m = np.maximum(s.max(axis=1, keepdims=True), 0.0)
        e = np.exp(s - m)
        out[:, h] = (e / (np.exp(-m) + e.sum(axis=1, keepdims=True))) @ v[:, h // per]
    return out


def keys_as_values_attention(X, W, p, m, rnd=same):
    """Attention whose values are the keys as they were before the rotation, with one added to the
    softmax's denominator and one logistic gate per head and token."""
    n, H, G, a = len(X), m["heads"], m["kv_heads"], m["dim"]
    q = rnd(X @ W[p + "q"].T).reshape(n, H, a)
    k = rnd(X @ W[p + "k"].T).reshape(n, G, a)
    qr, kr = (rnd(rotate_halves(z, range(n), m.get("rot"))) for z in (q, k))
    o = rnd(softmax_plus_one(qr, kr, k, m["scale"]))
    o = o * sigmoid(rnd(X @ W[p + "g"].T))[:, :, None]
    return rnd(o).reshape(n, H * a) @ W[p + "o"].T


# ---------------------------------------------------------------------------- gated delta rule
def causal_conv(x, w):
    """x [n, c], w [c, taps]: y_t = sum_j w[:, taps-1-j] x_(t-j), zeros before t = 0."""
    n, taps = len(x), w.shape[1]
    y = np.zeros(x.shape)
    for j in range(min(taps, n)):
        y[j:] += x[:n - j] * w[:, taps - 1 - j]
    return y


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def delta_memory(q, k, v, decay, beta):
    """q, k [n, H, a], v [n, H, b], decay and beta [n, H] -> [n, H, b]. A head's memory S [a, b]
    starts at zero; a token shrinks it, reads what its key finds, writes beta times the difference
    to its value back under the key, and then its query reads."""
    n, H, a = q.shape
    S = np.zeros((H, a, v.shape[2]))
    out = np.zeros(v.shape)
    for t in range(n):
        S *= decay[t][:, None, None]
        found = np.einsum("hab,ha->hb", S, k[t])
        S += k[t][:, :, None] * (beta[t][:, None] * (v[t] - found))[:, None, :]
        out[t] = np.einsum("hab,ha->hb", S, q[t])
    return out


def delta_mixer(X, W, p, m, eps, rnd=same):
    n, H, G, a, b = len(X), m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def stream(name, heads, size):
        return rnd(silu(causal_conv(rnd(X @ W[p + name].T), W[p + name + ".conv"]))).reshape(n, heads, size)

    q = np.repeat(unit(stream("q", G, a)) / math.sqrt(a), H // G, axis=1)
    k = np.repeat(unit(stream("k", G, a)), H // G, axis=1)
    beta = sigmoid(rnd(X @ W[p + "b"].T))
    decay = np.exp(-np.exp(W[p + "A_log"]) * softplus(rnd(X @ W[p + "a"].T) + W[p + "dt_bias"]))
    o = delta_memory(q, k, stream("v", H, b), decay, beta)
    o = rms_norm(o, W[p + "norm"], eps) * silu(rnd(X @ W[p + "g"].T)).reshape(n, H, b)
    return rnd(o).reshape(n, H * b) @ W[p + "o"].T


# ------------------------------------------------------------------------------ feed-forward
def plain(X, W, p, rnd=same):
    return rnd(relu_squared(rnd(X @ W[p + "up"].T))) @ W[p + "down"].T


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def choose_experts(s, correction, top, groups, keep):
    """One token's scores s [E] -> the chosen experts. The choice goes by s + correction; the
    experts fall into `groups` runs of neighbours, a run counts as its largest choice score, and
    all but the best `keep` runs are out (ties: the lower index)."""
    choice = s + correction
    size = len(s) // groups
    strength = choice.reshape(groups, size).max(axis=1)
    best = sorted(range(groups), key=lambda g: (-strength[g], g))[:keep]
    open_to = [e for e in range(len(s)) if e // size in best]
    return sorted(open_to, key=lambda e: (-choice[e], e))[:top]


def choice_margin(s, correction, top, groups, keep):
    """How far the choice of one token is from another one: the smaller of the gap between the
    weakest open group and the strongest closed one and of the gap between the last expert
    chosen and the next (infinite where nothing is left out)."""
    choice = s + correction
    runs = choice.reshape(groups, -1)
    order = np.argsort(-runs.max(axis=1), kind="stable")
    strength = runs.max(axis=1)[order]
    gap = strength[keep - 1] - strength[keep] if keep < groups else math.inf
    inside = np.sort(runs[order[:keep]].ravel())[::-1]
    return min(gap, inside[top - 1] - inside[top] if len(inside) > top else math.inf)


def routed(X, W, p, mlp, rnd=same, margins=None):
    r = mlp["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    s = softmax(X @ W[p + "router"].T)
    out = np.zeros(X.shape)
    for t in range(len(X)):
        if margins is not None:
            margins[t] = min(margins[t], choice_margin(s[t], W[p + "correction"], r["top"], g["count"], g["keep"]))
        for e in choose_experts(s[t], W[p + "correction"], r["top"], g["count"], g["keep"]):
            out[t] += s[t, e] * plain(X[t:t + 1], W, f"{p}e{e}.", rnd)[0]
    return out


# ------------------------------------------------------------------------------------- model
def run_order(cfg):
    """[(layer, whether the embedding output joins the stream ahead of it)] of a whole pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop = loop["start"], loop["stop"]
    out = [(i, False) for i in range(start)]
    for turn in range(loop["times"]):
        out += [(i, turn > 0 and i == start) for i in range(start, stop)]
    return out + [(i, False) for i in range(stop, n)]


def forward(cfg, W, tokens, layer_outputs=None, rnd=same, margins=None):
    """Logits [n, vocab] of a whole sequence. `layer_outputs`, a list, gets the stream after every
    layer run; `margins`, a list, gets for every token the closest call of any of its routers. With
    `rnd` (a rounding to a 16-bit type) the sublayers' inputs, the projections' results and what the
    last products read are rounded, as a 16-bit engine stores them; the stream, the norms, the
    softmax, the router and the recurrence stay."""
    eps = cfg["norm"]["eps"]
    first = rms_norm(W["embed"][np.asarray(tokens)].astype(np.float64), W["embed.norm"], eps)
    x = first.copy()
    if margins is not None:
        margins[:] = [math.inf] * len(x)
    for i, again in run_order(cfg):
        layer = cfg["layers"][i]
        p, m = f"l{i}.", layer["mixer"]
        if again:
            x = x + first
        h = rnd(rms_norm(x, W[p + "norm1"], eps))
        if layer["type"] == "delta":
            y = delta_mixer(h, W, p + "mix.", m, eps, rnd)
        else:
            y = keys_as_values_attention(h, W, p + "mix.", m, rnd)
        x = x + rms_norm(y, W[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rnd(rms_norm(x, W[p + "norm2"], eps))
            y = plain(h, W, p + "mlp.", rnd) if mlp["kind"] == "dense" else \
                routed(h, W, p + "mlp.", mlp, rnd, margins)
            x = x + rms_norm(y, W[p + "norm2b"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return rnd(rms_norm(x, W["final.norm"], eps)) @ W["head"].T


def greedy(cfg, W, prompt, n):
    """The n tokens that follow `prompt` when the largest logit is taken every time (ties: the
    lower id)."""
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(np.argmax(forward(cfg, W, seq)[-1]))
        out.append(tok)
        seq.append(tok)
    return out
