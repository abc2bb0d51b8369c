"""Small Bekunex configurations with weights of the tests' own making.

  B1: every size different from every other: a layer that makes a latent and reads it through a
      window of 13 (experts in four groups of three), a scan without a feed-forward, a layer that
      reads the first one's latent through a WIDER window than its own, rotated latent attention
      (experts in one group, no shared one), a second scan, a layer that reads the first latent
      through a narrower window.
  B2: the values a model may happen to make equal or 1: one head, a latent as wide as the model,
      key size = value size, a rotated part of one pair, a window of 1, one tap, one state, a step
      rank of 1, as many channels inside as outside, groups of a single expert, top 1, no factors.
  B3: scan layers only: no layer owns a paged cache; more states than 32 a channel.
  B4: sizes that no kernel's fast form takes (a width, head sizes, latents, channels and a
      vocabulary that are not multiples of 8); more states than 128 a channel; a layer without
      positions that reads the latent of a rotated one and does not know its rotated part.
  B5: sizes the tensor-core attention takes, more heads than a single-token tile of 16 rows in one
      layer and fewer in the other, a window longer than a key tile.
  B6: latent rows wider than 128 (the tensor-core kernels whose key tiles serve as values), with a
      window and a sink, more heads than one of their tiles has rows in one layer and three in
      the other.
"""
from __future__ import annotations

import copy

import numpy as np

from derosun_tiny import bf16_values, bind_model, write_model_dir  # noqa: F401
from plain_bekunex import choice_margin


def _lat(H, dim, rot, vdim, rank, base, scale):
    return {"type": "latent_attention",
            "mixer": {"heads": H, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                      "rot": {"dims": rot, "base": base}, "scale": scale}}


def _win(H, dim, vdim, rank, window, scale, lender=None):
    m = {"heads": H, "dim": dim, "vdim": vdim, "kv_rank": rank, "mask": {"size": window}, "scale": scale}
    if lender is not None:
        m["kv_from"] = lender
    return {"type": "latent_attention_2", "mixer": m}


def _scan(inner, state, rank, conv):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": rank, "conv": conv}}


def _moe(E, top, ff, count, keep, scale, shared):
    r = {"experts": E, "top": top, "scale": scale}
    if count:
        r["groups"] = {"count": count, "keep": keep}
    out = {"kind": "moe", "router": r, "expert": {"ff": ff}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def _model(vocab, width, eps, logit_scale, layers):
    return {"architecture": "Bekunex", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "logit_scale": logit_scale, "layers": [dict(layer, mlp=mlp) for layer, mlp in layers]}


B1 = _model(89, 48, 1e-5, 0.5, [
    (_win(3, 12, 20, 28, 13, 0.3), _moe(12, 3, 24, 4, 2, 2.5, 40)),
    (_scan(72, 5, 7, 4), None),
    (_win(5, 8, 6, 28, 30, 0.35, lender=0), _moe(6, 2, 32, 2, 1, 1.2, 16)),
    (_lat(4, 10, 6, 14, 20, 50.0, 0.25), _moe(5, 2, 28, 0, 0, 0.8, 0)),
    (_scan(40, 24, 3, 2), _moe(9, 4, 20, 3, 2, 1.7, 36)),
    (_win(2, 16, 10, 28, 4, 0.2, lender=0), None),
])

B2 = _model(70, 40, 1e-6, 1.0, [
    (_lat(1, 16, 2, 16, 40, 7.0, 0.3), _moe(4, 1, 40, 4, 2, 1.0, 40)),
    (_scan(40, 1, 1, 1), _moe(3, 1, 24, 1, 1, 1.0, 0)),
    (_win(1, 24, 24, 40, 1, 0.2), None),
    (_win(1, 24, 24, 40, 1, 0.2, lender=2), _moe(1, 1, 16, 1, 1, 1.0, 16)),
])

B3 = _model(50, 32, 1e-5, 2.0, [
    (_scan(56, 40, 5, 5), _moe(8, 3, 16, 2, 1, 2.0, 24)),
    (_scan(24, 12, 2, 3), None),
])

B4 = _model(53, 36, 1e-5, 0.7, [
    (_lat(5, 6, 4, 7, 11, 40.0, 0.4), _moe(10, 3, 20, 5, 3, 1.5, 12)),
    (_scan(42, 130, 3, 3), _moe(6, 2, 14, 3, 2, 0.6, 22)),
    (_win(3, 9, 5, 11, 19, 0.3, lender=0), None),
    (_win(7, 5, 3, 13, 6, 0.5), _moe(4, 2, 10, 2, 2, 3.0, 0)),
])

B5 = _model(96, 64, 1e-6, 0.25, [
    (_lat(20, 16, 16, 24, 48, 1000.0, 0.18), _moe(16, 4, 32, 4, 2, 2.0, 64)),
    (_win(4, 24, 16, 32, 90, 0.2), _moe(8, 2, 48, 2, 1, 1.5, 32)),
    (_scan(128, 16, 8, 4), _moe(8, 3, 16, 4, 2, 1.1, 24)),
    (_win(18, 8, 8, 32, 66, 0.3, lender=1), None),
])

B6 = _model(80, 64, 1e-6, 1.5, [
    (_win(72, 8, 8, 264, 40, 0.2), _moe(6, 2, 24, 3, 1, 1.5, 16)),
    (_lat(3, 16, 16, 24, 144, 1000.0, 0.18), None),
    (_scan(96, 32, 4, 4), _moe(4, 2, 16, 1, 1, 1.0, 0)),
    (_win(4, 16, 16, 144, 25, 0.25, lender=1), None),
])

CONFIGS = {"B1": (B1, 8), "B2": (B2, 16), "B3": (B3, 16), "B4": (B4, 4), "B5": (B5, 16),
           "B6": (B6, 16)}   # config, page size


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
    scores = (patterns @ router[:, :KINDS].T > 0) * 1.0
    for _ in range(20000):
        c = bf16_values(rng.uniform(-1.0, 1.0, E))
        if min(choice_margin(row, c, r["top"], g["count"], g["keep"]) for row in scores) > 0.03:
            return c
    raise ValueError("no corrections keep the choices apart")


def make_weights(cfg, seed):
    """name -> float64 array of bfloat16-exact values; lively enough that tokens differ, that
    corrections change which experts are chosen, that sinks and gates matter and that states
    decay at very different rates. Close calls between experts are rare: the first KINDS channels
    of the stream carry a sign per token that no layer writes over, every expert's logit is one
    of those channels, and the corrections keep the choices apart; so what a 16-bit
    engine rounds decides no choice, and which experts a token takes still depends on it."""
    rng = np.random.default_rng(seed)
    d, V = cfg["width"], cfg["vocab"]
    W = {}

    def mat(name, out, inp, gain=1.0):
        W[name] = rng.normal(0, gain / np.sqrt(inp), (out, inp))

    def vec(name, n, mean=0.0, sd=0.2):
        W[name] = mean + sd * rng.normal(0, 1, n)

    W["embed"] = rng.normal(0, 1.0, (V, d))
    W["embed"][:, :KINDS] = rng.choice([-3.0, 3.0], (V, KINDS)) * (1.0 + 0.05 * rng.normal(size=(V, KINDS)))
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        vec(p + "norm1", d, 1.0)
        vec(p + "norm1.b", d, 0.1, 0.3)
        W[p + "norm1"][:KINDS], W[p + "norm1.b"][:KINDS] = 1.0, 0.0
        p += "mix."
        if L["type"] == "mamba1":
            c, N, R = m["inner"], m["state"], m["dt_rank"]
            mat(p + "in", 2 * c, d, 1.5)
            W[p + "conv"] = rng.normal(0, 0.6, (c, m["conv"]))
            vec(p + "conv.b", c)
            mat(p + "x", R + 2 * N, c, 1.5)
            mat(p + "dt", c, R)
            vec(p + "dt.b", c, -1.5, 1.0)
            W[p + "A_log"] = rng.normal(-1.0, 1.5, (c, N))
            vec(p + "D", c, 0.5, 0.5)
            mat(p + "o", d, c)
        else:
            H, dim, vdim, r, rot = m["heads"], m["dim"], m["vdim"], m["kv_rank"], m.get("rot_dim", 0)
            mat(p + "q", H * (dim + rot), d, 3.0)
            if m.get("kv_from") is None:
                mat(p + "dkv", r + rot, d, 2.0)
                vec(p + "dkv.norm", r, 1.5, 0.3)
            mat(p + "uk", H * dim, r, 1.5)
            mat(p + "uv", H * vdim, r)
            if L["type"] == "latent_attention_2":
                vec(p + "sink", H, 0.5, 1.0)
                mat(p + "g", H * vdim, d, 2.0)
            mat(p + "o", d, H * vdim)
        mlp = L.get("mlp")
        if mlp:
            p = f"l{i}.mlp."
            E, f = mlp["router"]["experts"], mlp["expert"]["ff"]
            W[p + "router"] = np.zeros((E, d))
            for e in range(E):
                W[p + "router"][e, rng.integers(KINDS)] = rng.choice([-8.0, 8.0])
            W[p + "correction"] = apart(rng, W[p + "router"], mlp["router"])
            for e in range(E):
                mat(f"{p}e{e}.gate", f, d, 1.5)
                mat(f"{p}e{e}.up", f, d)
                mat(f"{p}e{e}.down", d, f)
            if mlp.get("shared"):
                f = mlp["shared"]["ff"]
                mat(p + "shared.gate", f, d, 1.5)
                mat(p + "shared.up", f, d)
                mat(p + "shared.down", d, f)
    for name in W:
        if name.endswith(("mix.o", ".down")):
            W[name][:KINDS] = 0.0
    vec("final.norm", d, 1.0)
    vec("final.norm.b", d, 0.0, 0.3)
    mat("head", V, d, 2.0)
    return {k: bf16_values(v) for k, v in W.items()}
