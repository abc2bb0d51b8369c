"""Small Kesozen configurations with weights of the tests' own making.

  K1: every size different from every other: a layer before the loop, three looped layers (delta,
      attention, delta without a feed-forward) three times, two after it; values wider and narrower
      than keys, several value heads a key head, experts in groups with and without a loser, dense
      feed-forwards.
  K2: the values a model may happen to make equal or 1: one head, one tap, one expert, groups of a
      single expert, top 1, a whole-head rotation, a loop run once over every layer.
  K3: delta layers only (no layer owns a paged cache), a loop of one layer, odd key sizes.
  K4: sizes that no kernel's fast form takes: a width, head sizes and a vocabulary that are not
      multiples of 4; more taps than a portion has tokens; no rotation, no loop.
  K5: sizes the tensor-core attention takes, more heads than a single-token tile of 16 rows in one
      layer and fewer in the other; keys of 128 and more channels in the delta layers.
"""
from __future__ import annotations

import copy

import numpy as np

from derosun_tiny import bf16_values, bind_model, write_model_dir  # noqa: F401
from plain_kesozen import choice_margin, softmax


def _att(H, G, dim, rot, base, scale):
    m = {"heads": H, "kv_heads": G, "dim": dim, "vdim": dim, "scale": scale}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
    return {"type": "attention", "mixer": m}


def _delta(H, G, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": H, "kv_heads": G, "dim": dim, "vdim": vdim, "conv": conv}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(E, top, ff, count=0, keep=0):
    r = {"experts": E, "top": top}
    if count:
        r["groups"] = {"count": count, "keep": keep}
    return {"kind": "moe", "router": r, "expert": {"ff": ff}}


def _model(vocab, width, eps, loop, layers):
    out = {"architecture": "Kesozen", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "layers": [dict(layer, mlp=mlp) for layer, mlp in layers]}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


K1 = _model(89, 48, 1e-2, (1, 4, 3), [
    (_att(6, 3, 20, 12, 300.0, 0.3), _dense(56)),
    (_delta(4, 2, 12, 24, 4), _moe(12, 3, 24, 4, 2)),
    (_att(4, 1, 16, 4, 50.0, 0.35), _moe(10, 4, 28, 5, 3)),
    (_delta(3, 3, 36, 8, 3), None),
    (_att(2, 2, 28, 28, 9000.0, 0.25), None),
    (_delta(6, 2, 8, 20, 2), _moe(7, 2, 32)),
])

K2 = _model(70, 40, 1e-6, (0, 3, 1), [
    (_delta(1, 1, 16, 16, 1), _moe(4, 1, 40, 4, 2)),
    (_att(1, 1, 40, 40, 7.0, 0.2), _moe(1, 1, 24, 1, 1)),
    (_delta(1, 1, 1, 4, 2), _dense(40)),
])

K3 = _model(50, 32, 1e-5, (1, 2, 4), [
    (_delta(4, 4, 13, 10, 5), _moe(8, 3, 16, 2, 1)),
    (_delta(2, 1, 7, 12, 3), _dense(24)),
    (_delta(3, 1, 40, 33, 2), None),
])

K4 = _model(53, 37, 1e-3, None, [
    (_att(5, 5, 11, 6, 40.0, 0.4), _moe(9, 3, 21, 3, 2)),
    (_delta(3, 1, 9, 7, 9), _dense(27)),
    (_att(6, 2, 9, 0, 0.0, 0.5), _moe(6, 6, 14, 2, 2)),
])

K5 = _model(96, 64, 1e-6, (0, 2, 2), [
    (_att(20, 1, 32, 16, 1000.0, 0.2), _moe(16, 4, 32, 4, 2)),
    (_delta(4, 2, 128, 64, 4), _moe(8, 2, 48, 4, 1)),
    (_att(8, 2, 64, 48, 100.0, 0.15), _dense(96)),
    (_delta(2, 2, 144, 128, 3), _moe(8, 3, 16, 2, 1)),
    (_delta(2, 1, 64, 256, 4), None),
])

CONFIGS = {"K1": (K1, 8), "K2": (K2, 16), "K3": (K3, 16), "K4": (K4, 4), "K5": (K5, 16)}   # config, page size


def changed(cfg, path, value):
    """A copy of cfg with the value at `path` replaced (... takes the key out)."""
    cfg = copy.deepcopy(cfg)
    at = cfg
    for key in path[:-1]:
        at = at[key]
    if value is ...:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return cfg


KINDS = 6


def apart(rng, router, r):
    """Corrections with which no choice is close, whatever the signs of the KINDS channels."""
    E, g = r["experts"], r.get("groups") or {"count": 1, "keep": 1}
    patterns = np.array(np.meshgrid(*[[-1.0, 1.0]] * KINDS)).reshape(KINDS, -1).T
    for spread in (0.6, 1.0, 2.0, 4.0):
        for _ in range(2000):
            c = bf16_values(rng.uniform(-spread, spread, E))
            near = min(choice_margin(softmax(a * row), c, r["top"], g["count"], g["keep"])
                       for row in patterns @ router[:, :KINDS].T for a in (0.4, 0.6, 0.8, 1.0, 1.3, 1.7, 2.2))
            if near > 0.02:
                return c
    raise ValueError("no corrections keep the choices apart")


def make_weights(cfg, seed):
    """name -> float64 array of bfloat16-exact values; lively enough that tokens differ, that the
    correction changes which experts are chosen, that gates and the added one matter and that
    memories decay at very different rates. Close calls between experts are rare: the first KINDS
    channels of the stream carry a sign per token that no layer writes over, every expert's logit is
    one of those channels, and the corrections keep the choices apart; so what a 16-bit engine rounds
    decides no choice, and which experts a token takes still depends on it."""
    rng = np.random.default_rng(seed)
    d, V = cfg["width"], cfg["vocab"]
    W = {}

    def mat(name, out, inp, gain=1.0):
        W[name] = rng.normal(0, gain / np.sqrt(inp), (out, inp))

    def vec(name, n, mean=0.0, sd=0.2):
        W[name] = mean + sd * rng.normal(0, 1, n)

    W["embed"] = rng.normal(0, 1.0, (V, d))
    W["embed"][:, :KINDS] = rng.choice([-1.5, 1.5], (V, KINDS))
    vec("embed.norm", d, 1.2)
    W["embed.norm"][:KINDS] = 1.0
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        mlp = L.get("mlp")
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp else ()):
            vec(p + name, d, 0.5 if name.endswith("b") else 1.0)
            W[p + name][:KINDS] = 0.0 if name.endswith("b") else 1.0
        p += "mix."
        H, G, dim = m["heads"], m["kv_heads"], m["dim"]
        if L["type"] == "delta":
            vdim = m["vdim"]
            for name, rows in (("q", G * dim), ("k", G * dim), ("v", H * vdim)):
                mat(p + name, rows, d, 1.5)
                W[f"{p}{name}.conv"] = rng.normal(0, 0.7, (rows, m["conv"]))
            mat(p + "a", H, d, 1.5)
            mat(p + "b", H, d, 1.5)
            vec(p + "dt_bias", H, -1.0, 1.0)
            W[p + "A_log"] = rng.normal(-1.0, 1.5, H)
            vec(p + "norm", vdim, 1.0, 0.3)
            mat(p + "g", H * vdim, d, 1.5)
            mat(p + "o", d, H * vdim)
        else:
            mat(p + "q", H * dim, d, 2.5)
            mat(p + "k", G * dim, d, 1.5)
            mat(p + "g", H, d, 2.0)
            mat(p + "o", d, H * dim)
        if not mlp:
            continue
        p = f"l{i}.mlp."
        if mlp["kind"] == "dense":
            mat(p + "up", mlp["ff"], d, 1.5)
            mat(p + "down", d, mlp["ff"])
            continue
        E, f = mlp["router"]["experts"], mlp["expert"]["ff"]
        W[p + "router"] = np.zeros((E, d))
        for e in range(E):
            W[p + "router"][e, rng.integers(KINDS)] = rng.choice([-2.0, 2.0])
        W[p + "correction"] = apart(rng, W[p + "router"], mlp["router"])
        for e in range(E):
            mat(f"{p}e{e}.up", f, d, 1.5)
            mat(f"{p}e{e}.down", d, f)
    vec("final.norm", d, 1.0)
    mat("head", V, d, 2.0)
    return {k: bf16_values(v) for k, v in W.items()}
