"""Typed reading of a Kesozen config.json, and its translation to a ModelSpec.

Kesozen is a decoder whose layers are listed one by one in the file. A layer norms the input AND the
output of each sublayer:

    x <- x + norm1b(mixer(norm1(x)));  x <- x + norm2b(feed_forward(norm2(x)))

The embedding rows are normed too. With `loop` {start, stop, times} the layers start .. stop - 1 run
`times` times in a row with the same weights and a cache or state of their own each time; ahead of
every time but the first the embedding output joins the stream once more.

Its mixers: "attention", causal grouped-query attention with a half-split rotation of part of every
head, whose values are the keys before the rotation, with one added to the softmax's denominator and
a logistic gate on each head; "delta", a gated delta rule with a 32-bit state per request. Its
feed-forwards: W_down relu(W_up x)^2, a mixture of such experts (softmax scores over all experts,
chosen by score + correction inside the best groups of experts, a group counting as its largest
choice score, weights not renormalized), or none. The head has a matrix of its own.

Every size and constant comes from the file; a value the engine cannot honour is refused with its
key in the message.
"""
from __future__ import annotations

from typing import Optional

from .derosun import _rotation, _scale
from .gafonex import _int, _positive
from .qwen3 import ConfigError
from .spec import FeedForwardSpec, LayerCall, LayerSpec, MixerSpec, ModelSpec, NormSpec
from .totatar import _object

ARCHITECTURE = "Kesozen"

ATTENTION_TENSORS = (("q", "mix.q"), ("k", "mix.k"), ("gate", "mix.g"), ("o", "mix.o"))
DELTA_TENSORS = (("q", "mix.q"), ("k", "mix.k"), ("v", "mix.v"), ("q_conv", "mix.q.conv"),
                 ("k_conv", "mix.k.conv"), ("v_conv", "mix.v.conv"), ("a", "mix.a"), ("b", "mix.b"),
                 ("gate", "mix.g"), ("a_log", "mix.A_log"), ("dt_bias", "mix.dt_bias"), ("norm", "mix.norm"),
                 ("o", "mix.o"))
DENSE_TENSORS = (("up", "mlp.up"), ("down", "mlp.down"))
ROUTED_TENSORS = (("expert_up", "mlp.e{e}.up"), ("expert_down", "mlp.e{e}.down"), ("router", "mlp.router"),
                  ("router_correction", "mlp.correction"))
BLOCK_TENSORS = (("mixer_norm", "norm1"), ("mixer_out_norm", "norm1b"), ("ffn_norm", "norm2"),
                 ("ffn_out_norm", "norm2b"))


def _heads(m: dict, where: str) -> tuple:
    H = _int(m, "heads", where)
    G = _int(m, "kv_heads", where, default=H)
    if H % G:
        raise ConfigError(f"config: {where}heads ({H}) is not a multiple of kv_heads ({G})")
    return H, G


def _attention(m: dict, where: str, eps: float) -> MixerSpec:
    H, G = _heads(m, where)
    dim = _int(m, "dim", where)
    vdim = _int(m, "vdim", where, default=dim)
    if vdim != dim:
        raise ConfigError(f"config: {where}vdim is {vdim}; the values are the keys, so it must be dim ({dim})")
    return MixerSpec("sink_attention", num_heads=H, num_kv_heads=G, head_dim=dim, value_dim=dim,
                     scale=_scale(m, where), sink_score=0.0, values_from_keys=True, output_gate=True,
                     gate_activation="sigmoid", gate_scope="head", norm_eps=eps, tensors=ATTENTION_TENSORS,
                     position=_rotation(m.get("rot"), dim, where, "rope_half_split", ()))


def _delta(m: dict, where: str, eps: float) -> MixerSpec:
    H, G = _heads(m, where)
    dim, taps = _int(m, "dim", where), _int(m, "conv", where)
    if dim > 256:
        raise ConfigError(f"config: {where}dim is {dim}; the delta rule takes keys of at most 256")
    if taps > 64:
        raise ConfigError(f"config: {where}conv is {taps}; the convolution takes at most 64 taps")
    return MixerSpec("gated_delta", num_heads=H, num_kv_heads=G, head_dim=dim,
                     value_dim=_int(m, "vdim", where, default=dim), conv_taps=taps, norm_eps=eps,
                     tensors=DELTA_TENSORS)


MIXER_READERS = {"attention": _attention, "delta": _delta}


def _feed_forward(mlp, where: str) -> Optional[FeedForwardSpec]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config: {where}mlp must be an object or null")
    where += "mlp."
    kind = mlp.get("kind")
    if kind == "dense":
        return FeedForwardSpec("plain_dense", intermediate_size=_int(mlp, "ff", where), tensors=DENSE_TENSORS,
                               activation="relu_squared")
    if kind != "moe":
        raise ConfigError(f"config: {where}kind is {kind!r}; known kinds: dense, moe")
    router = _object(mlp, "router", where)
    at = where + "router."
    E, top = _int(router, "experts", at), _int(router, "top", at)
    if top > E or top > 32:
        raise ConfigError(f"config: {at}top is {top}; at most the number of experts ({E}) and at most 32")
    if E > 2048:
        raise ConfigError(f"config: {at}experts is {E}; the router takes at most 2048")
    groups = _object(router, "groups", at, required=False)
    count = keep = 1
    if groups is not None:
        count, keep = _int(groups, "count", at + "groups."), _int(groups, "keep", at + "groups.")
        if E % count:
            raise ConfigError(f"config: {at}groups.count is {count}; it must divide the {E} experts")
        if keep > count or keep * (E // count) < top:
            raise ConfigError(f"config: {at}groups.keep is {keep}; at most the {count} groups, and enough of "
                              f"them to hold the top {top}")
    expert = _object(mlp, "expert", where)
    return FeedForwardSpec("routed_experts", intermediate_size=_int(expert, "ff", where + "expert."),
                           tensors=ROUTED_TENSORS, activation="relu_squared", experts=E, top=top, gated=False,
                           router_scores="all", router_correction=True, router_renormalize=False,
                           router_groups=(count, keep), router_group_best=1)


def _run_order(raw: dict, n: int) -> list:
    """The calls of one pass over `n` layers: as listed, with the looped ones repeated."""
    loop = _object(raw, "loop", "", required=False)
    if loop is None:
        return [LayerCall(i) for i in range(n)]
    start, times = loop.get("start"), _int(loop, "times", "loop.")
    if isinstance(start, bool) or not isinstance(start, int) or start < 0:
        raise ConfigError(f"config: loop.start is {start!r}; it must be the number of a layer")
    stop = _int(loop, "stop", "loop.")
    if not start < stop <= n:
        raise ConfigError(f"config: loop.stop is {stop}; it must be beyond loop.start ({start}) and at most "
                          f"the number of layers ({n})")
    calls = [LayerCall(i) for i in range(start)]
    for turn in range(times):
        calls += [LayerCall(i, adds_embedding=turn > 0 and i == start) for i in range(start, stop)]
    return calls + [LayerCall(i) for i in range(stop, n)]


def kesozen_model_spec(raw: dict) -> ModelSpec:
    """config.json (as a dict) -> ModelSpec. Tensor names: `embed` and `embed.norm`, `l<i>.norm1`,
    `.norm1b`, `.norm2`, `.norm2b`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`."""
    if not isinstance(raw, dict):
        raise ConfigError("config: the top level must be an object")
    d = _int(raw, "width", "")
    V = _int(raw, "vocab", "")
    norm = raw.get("norm")
    if not isinstance(norm, dict):
        raise ConfigError("config: norm is required (eps)")
    eps = _positive(norm, "eps", "norm.")
    nspec = NormSpec("rmsnorm", eps)
    entries = raw.get("layers")
    if not isinstance(entries, list) or not entries:
        raise ConfigError("config: layers must list at least one layer")
    layers = []
    for i, e in enumerate(entries):
        where = f"layers[{i}]."
        if not isinstance(e, dict) or not isinstance(e.get("mixer"), dict):
            raise ConfigError(f"config: {where}mixer is required")
        kind = e.get("type")
        if kind not in MIXER_READERS:
            raise ConfigError(f"config: {where}type is {kind!r}; known mixers are "
                              + ", ".join(sorted(MIXER_READERS)))
        mixer = MIXER_READERS[kind](e["mixer"], where + "mixer.", eps)
        layers.append(LayerSpec("sandwich_norm_residual", f"l{i}.", mixer, _feed_forward(e.get("mlp"), where),
                                nspec, BLOCK_TENSORS))
    spec = ModelSpec(
        architecture=ARCHITECTURE, hidden_size=d, vocab_size=V, layers=layers,
        run_order=_run_order(raw, len(layers)), final_norm=nspec, embedding_name="embed",
        final_norm_name="final.norm", head_name="head", embedding_norm=nspec,
        embedding_norm_name="embed.norm", source=dict(raw))
    spec.validate()
    return spec
