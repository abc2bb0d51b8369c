"""Typed reading of a Bekunex config.json, and its translation to a ModelSpec.

Bekunex is a decoder whose layers are listed one by one in the file. Both sublayers of a layer
read one layer norm (with a bias) and are added to the stream together:

    n = norm1(x);  x <- x + (mixer(n) + feed_forward(n))

Its mixers: "latent_attention", causal attention over one small cached latent per token with a
rotated key part that all heads share, queries straight from the layer's input;
"latent_attention_2", the same without positions, with a sliding window, a sink per head and a
logistic gate on the heads, whose latent may be that of an earlier layer (`kv_from`); "mamba1", a
selective scan with a decay per channel and state and a 32-bit state per request. Its
feed-forward is a mixture of SiLU-gated experts with a shared one, chosen by logistic scores with
a correction inside the best groups of experts, or absent. The head has a matrix of its own; the
logits are multiplied by `logit_scale`.

Every size and constant comes from the file; a value the engine cannot honour is refused with its
key in the message.
"""
from __future__ import annotations

from typing import Optional

from .derosun import _rotation, _scale
from .gafonex import _int, _number, _positive
from .qwen3 import ConfigError
from .spec import FeedForwardSpec, LayerCall, LayerSpec, MixerSpec, ModelSpec, NormSpec
from .totatar import _object

ARCHITECTURE = "Bekunex"

LATENT_TENSORS = (("q", "mix.q"), ("kv_down", "mix.dkv"), ("kv_norm", "mix.dkv.norm"),
                  ("k_up", "mix.uk"), ("v_up", "mix.uv"), ("sink", "mix.sink"), ("gate", "mix.g"),
                  ("o", "mix.o"))
SCAN_TENSORS = (("in", "mix.in"), ("conv", "mix.conv"), ("conv_bias", "mix.conv.b"), ("x", "mix.x"),
                ("dt", "mix.dt"), ("dt_bias", "mix.dt.b"), ("a_log", "mix.A_log"), ("d", "mix.D"),
                ("o", "mix.o"))
ROUTED_TENSORS = (("expert_gate", "mlp.e{e}.gate"), ("expert_up", "mlp.e{e}.up"),
                  ("expert_down", "mlp.e{e}.down"), ("router", "mlp.router"),
                  ("router_correction", "mlp.correction"))
SHARED_TENSORS = (("gate", "mlp.shared.gate"), ("up", "mlp.shared.up"), ("down", "mlp.shared.down"))
BLOCK_TENSORS = (("mixer_norm", "norm1"),)


def _latent_sizes(m: dict, where: str, eps: float) -> dict:
    dim = _int(m, "dim", where)
    return {"num_heads": _int(m, "heads", where), "num_kv_heads": 1, "head_dim": dim,
            "value_dim": _int(m, "vdim", where, default=dim), "latent_rank": _int(m, "kv_rank", where),
            "norm_eps": eps, "scale": _scale(m, where), "tensors": LATENT_TENSORS}


def _latent_attention(m: dict, where: str, eps: float, lender: Optional[MixerSpec]) -> MixerSpec:
    rot_dim = _int(m, "rot_dim", where)
    return MixerSpec("latent_attention", rope_dim=rot_dim,
                     position=_rotation(m.get("rot"), rot_dim, where, "rope_half_split", ()),
                     **_latent_sizes(m, where, eps))


def _latent_attention_2(m: dict, where: str, eps: float, lender: Optional[MixerSpec]) -> MixerSpec:
    sizes = _latent_sizes(m, where, eps)
    mask = _object(m, "mask", where, required=False)
    window = _int(mask, "size", where + "mask.") if mask is not None else None
    row = 0
    if lender is not None:
        if lender.latent_rank != sizes["latent_rank"]:
            raise ConfigError(f"config: {where}kv_rank is {sizes['latent_rank']}; the layer whose latent "
                              f"it reads (kv_from) has {lender.latent_rank}")
        row = lender.latent_rank + lender.rope_dim
    return MixerSpec("latent_attention", window=window, sink=True, output_gate=True,
                     gate_activation="sigmoid", borrows_latent=lender is not None, cache_row=row, **sizes)


def _mamba1(m: dict, where: str, eps: float, lender: Optional[MixerSpec]) -> MixerSpec:
    N = _int(m, "state", where)
    if N > 256:
        raise ConfigError(f"config: {where}state is {N}; the scan keeps at most 256 per channel")
    taps = _int(m, "conv", where)
    if taps > 64:
        raise ConfigError(f"config: {where}conv is {taps}; the convolution takes at most 64 taps")
    return MixerSpec("channel_state_space", inner_dim=_int(m, "inner", where), head_dim=N,
                     dt_rank=_int(m, "dt_rank", where), conv_taps=taps, tensors=SCAN_TENSORS)


MIXER_READERS = {"latent_attention": _latent_attention, "latent_attention_2": _latent_attention_2,
                 "mamba1": _mamba1}


def _lender(m: dict, where: str, i: int, kind: str, layers: list) -> Optional[int]:
    """The earlier layer whose latent a mixer reads (`kv_from`), or None."""
    if m.get("kv_from") is None:
        return None
    if kind != "latent_attention_2":
        raise ConfigError(f"config: {where}kv_from belongs to latent_attention_2")
    j = m["kv_from"]
    if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < i:
        raise ConfigError(f"config: {where}kv_from is {j!r}; it must name an earlier layer")
    lender = layers[j].mixer
    if lender.kind != "latent_attention" or lender.borrows_latent:
        raise ConfigError(f"config: {where}kv_from is {j}, a layer without a latent of its own")
    return j


def _feed_forward(mlp, where: str) -> Optional[FeedForwardSpec]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config: {where}mlp must be an object or null")
    where += "mlp."
    kind = mlp.get("kind")
    if kind != "moe":
        raise ConfigError(f"config: {where}kind is {kind!r}; known kinds: moe")
    router = _object(mlp, "router", where)
    E, top = _int(router, "experts", where + "router."), _int(router, "top", where + "router.")
    if top > E or top > 32:
        raise ConfigError(f"config: {where}router.top is {top}; at most the number of experts ({E}) "
                          "and at most 32")
    if E > 2048:
        raise ConfigError(f"config: {where}router.experts is {E}; the router takes at most 2048")
    groups = _object(router, "groups", where + "router.", required=False)
    count = keep = 1
    if groups is not None:
        count = _int(groups, "count", where + "router.groups.")
        keep = _int(groups, "keep", where + "router.groups.")
        if E % count:
            raise ConfigError(f"config: {where}router.groups.count is {count}; it must divide the "
                              f"{E} experts")
        if keep > count or keep * (E // count) < top:
            raise ConfigError(f"config: {where}router.groups.keep is {keep}; at most the {count} groups, "
                              f"and enough of them to hold the top {top}")
    scale = _number(router, "scale", where + "router.") if router.get("scale") is not None else 1.0
    shared = _object(mlp, "shared", where, required=False)
    shared_spec = None if shared is None else \
        FeedForwardSpec("gated_dense", intermediate_size=_int(shared, "ff", where + "shared."),
                        tensors=SHARED_TENSORS, activation="silu")
    expert = _object(mlp, "expert", where)
    return FeedForwardSpec("routed_experts", intermediate_size=_int(expert, "ff", where + "expert."),
                           tensors=ROUTED_TENSORS, activation="silu", experts=E, top=top,
                           shared=shared_spec, router_scores="sigmoid", router_correction=True,
                           router_renormalize=False, router_scale=scale, router_groups=(count, keep))


def bekunex_model_spec(raw: dict) -> ModelSpec:
    """config.json (as a dict) -> ModelSpec. Tensor names: `embed`, `l<i>.norm1` and `.b`,
    `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm` and `.b`, `head`."""
    if not isinstance(raw, dict):
        raise ConfigError("config: the top level must be an object")
    d = _int(raw, "width", "")
    V = _int(raw, "vocab", "")
    norm = raw.get("norm")
    if not isinstance(norm, dict):
        raise ConfigError("config: norm is required (eps)")
    eps = _positive(norm, "eps", "norm.")
    nspec = NormSpec("layernorm", eps, bias_suffix=".b")
    entries = raw.get("layers")
    if not isinstance(entries, list) or not entries:
        raise ConfigError("config: layers must list at least one layer")
    layers, calls = [], []
    for i, e in enumerate(entries):
        where = f"layers[{i}]."
        if not isinstance(e, dict) or not isinstance(e.get("mixer"), dict):
            raise ConfigError(f"config: {where}mixer is required")
        kind = e.get("type")
        if kind not in MIXER_READERS:
            raise ConfigError(f"config: {where}type is {kind!r}; known mixers are "
                              + ", ".join(sorted(MIXER_READERS)))
        j = _lender(e["mixer"], where + "mixer.", i, kind, layers)
        mixer = MIXER_READERS[kind](e["mixer"], where + "mixer.", eps,
                                    layers[j].mixer if j is not None else None)
        layers.append(LayerSpec("parallel_residual", f"l{i}.", mixer, _feed_forward(e.get("mlp"), where),
                                nspec, BLOCK_TENSORS))
        calls.append(LayerCall(i, cache_from=j))
    spec = ModelSpec(
        architecture=ARCHITECTURE, hidden_size=d, vocab_size=V, layers=layers, run_order=calls,
        final_norm=nspec, embedding_name="embed", final_norm_name="final.norm", head_name="head",
        logit_scale=_number(raw, "logit_scale", "") if raw.get("logit_scale") is not None else 1.0,
        source=dict(raw))
    spec.validate()
    return spec
