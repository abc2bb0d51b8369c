"""Bekunex without a GPU: the config reader and its refusals, the declared tensor names, the
plain statement's pieces against values worked out by hand, and the engine's host side (cache
groups with borrowed latents, state rows, packing, portions, mixed batches, reused pages and
slots) with torch stand-ins for the kernels, against the plain statement."""
import math

import numpy as np
import pytest
import torch

import bekunex_tiny as bt
import emulated_kernels
import plain_bekunex as plain
import tiny


def test_reader_builds_the_layers_the_file_lists():
    from tgo_b200.registry import model_spec_from_config
    spec = model_spec_from_config(bt.B1)
    assert spec.architecture == "Bekunex" and not spec.tied_head and len(spec.layers) == 6
    assert {ls.block for ls in spec.layers} == {"parallel_residual"}
    assert spec.logit_scale == 0.5 and spec.final_norm.kind == "layernorm"
    assert [c.cache_from for c in spec.run_order] == [None, None, 0, None, None, 0]
    win = spec.layers[0].mixer
    assert (win.kind, win.num_heads, win.head_dim, win.value_dim, win.latent_rank, win.window) == \
        ("latent_attention", 3, 12, 20, 28, 13)
    assert win.sink and win.output_gate and win.gate_activation == "sigmoid" and not win.borrows_latent
    assert win.rope_dim == 0 and win.query_rank == 0 and win.position is None and win.scale == 0.3
    lent = spec.layers[2].mixer
    assert lent.borrows_latent and lent.window == 30 and lent.cache_row == 28
    rot = spec.layers[3].mixer
    assert (rot.rope_dim, rot.window, rot.sink, rot.output_gate) == (6, None, False, False)
    assert rot.position.kind == "rope_half_split" and rot.position.theta == 50.0
    scan = spec.layers[1].mixer
    assert (scan.kind, scan.inner_dim, scan.head_dim, scan.dt_rank, scan.conv_taps) == \
        ("channel_state_space", 72, 5, 7, 4)
    assert spec.layers[1].feed_forward is None
    moe = spec.layers[0].feed_forward
    assert (moe.experts, moe.top, moe.intermediate_size, moe.router_groups, moe.router_scale) == \
        (12, 3, 24, (4, 2), 2.5)
    assert moe.router_scores == "sigmoid" and moe.router_correction and not moe.router_renormalize
    assert moe.shared.intermediate_size == 40 and not moe.router_bias
    assert spec.layers[3].feed_forward.router_groups == (1, 1) and spec.layers[3].feed_forward.shared is None
    assert model_spec_from_config(bt.changed(bt.B1, ("logit_scale",), ...)).logit_scale == 1.0
    # the latent of a rotated layer, read by one that knows no positions: rows with channels more
    assert model_spec_from_config(bt.B4).layers[2].mixer.cache_row == 11 + 4


@pytest.mark.parametrize("path,value,word", [
    (("width",), 0, "width"), (("vocab",), ..., "vocab"), (("norm", "eps"), -1.0, "norm.eps"),
    (("logit_scale",), "two", "logit_scale"), (("logit_scale",), float("inf"), "logit_scale"),
    (("layers", 0, "type"), "conv", "layers[0].type"),
    (("layers", 0, "mixer", "heads"), ..., "heads"), (("layers", 0, "mixer", "kv_rank"), 0, "kv_rank"),
    (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"), (("layers", 0, "mixer", "scale"), -1.0, "scale"),
    (("layers", 0, "mixer", "kv_from"), 0, "kv_from"), (("layers", 2, "mixer", "kv_from"), 1, "kv_from"),
    (("layers", 2, "mixer", "kv_from"), "0", "kv_from"), (("layers", 5, "mixer", "kv_from"), 2, "kv_from"),
    (("layers", 5, "mixer", "kv_from"), -1, "kv_from"), (("layers", 3, "mixer", "kv_from"), 0, "kv_from"),
    (("layers", 2, "mixer", "kv_rank"), 20, "kv_rank"),
    (("layers", 3, "mixer", "rot", "dims"), 5, "rot.dims"), (("layers", 3, "mixer", "rot", "base"), 0.0, "rot.base"),
    (("layers", 3, "mixer", "rot_dim"), ..., "rot_dim"),
    (("layers", 1, "mixer", "state"), 257, "state"), (("layers", 1, "mixer", "conv"), 65, "conv"),
    (("layers", 1, "mixer", "dt_rank"), ..., "dt_rank"), (("layers", 1, "mixer", "inner"), 1.5, "inner"),
    (("layers", 0, "mlp", "kind"), "dense", "mlp.kind"),
    (("layers", 0, "mlp", "router", "top"), 13, "router.top"),
    (("layers", 0, "mlp", "router", "groups", "count"), 5, "groups.count"),
    (("layers", 0, "mlp", "router", "groups", "keep"), 5, "groups.keep"),
    (("layers", 4, "mlp", "router", "groups", "keep"), 1, "groups.keep"),
    (("layers", 0, "mlp", "router", "scale"), "x", "router.scale"),
    (("layers", 0, "mlp", "expert", "ff"), ..., "expert.ff"), (("layers", 0, "mlp", "shared", "ff"), 0, "shared.ff"),
])
def test_reader_refuses_by_key(path, value, word):
    from tgo_b200.config.qwen3 import ConfigError
    from tgo_b200.registry import model_spec_from_config
    with pytest.raises(ConfigError) as err:
        model_spec_from_config(bt.changed(bt.B1, path, value))
    assert word in str(err.value)


@pytest.mark.parametrize("name", sorted(bt.CONFIGS))
def test_declared_tensors_are_the_weights_the_tests_make(name):
    from tgo_b200.engine.model import Model
    from tgo_b200.registry import model_spec_from_config
    cfg, _ = bt.CONFIGS[name]
    W = bt.make_weights(cfg, 1)
    model = Model(model_spec_from_config(cfg), torch.float32, "cpu")
    declared = {w.name: tuple(w.shape) for w in model.weight_specs() if not w.optional}
    assert declared == {k: tuple(v.shape) for k, v in W.items()}


def test_a_written_folder_loads(tmp_path):
    from tgo_b200.engine.model import Model
    from tgo_b200.registry import model_spec_from_config
    from tgo_b200.weights.binder import WeightError, load_weights
    from tgo_b200.weights.safetensors import SafetensorsRepo
    W = bt.make_weights(bt.B1, 2)
    d = bt.write_model_dir(str(tmp_path / "m"), bt.B1, W)
    model = Model(model_spec_from_config(bt.B1), torch.bfloat16, "cpu")
    weights = load_weights(model.weight_specs(), SafetensorsRepo(d), torch.bfloat16, "cpu", None, log=None)
    for name in ("l0.norm1.b", "l1.mix.A_log", "l1.mix.dt.b", "l0.mix.sink", "l0.mlp.correction", "final.norm.b"):
        assert weights[name].dtype == torch.float32, name
    model.bind(dict(weights))
    # q, the cached row and the gate are one product; a borrowing layer's has no row to cache
    assert model.blocks[0].mixer.w_in.shape == (3 * 12 + 28 + 3 * 20, 48)
    assert model.blocks[2].mixer.w_in.shape == (5 * 8 + 5 * 6, 48)
    # the step sizes' matrix reads r | B | C as they lie, with zeros over B and C
    scan = model.blocks[1].mixer
    assert scan.w_x.shape == (24, 72) and scan.w_dt.shape == (72, 24)
    assert not scan.w_dt[:, 7:].any() and not scan.w_x[17:].any()
    # the factor on the logits lies in the final norm
    assert torch.allclose(model.final_norm.gain, torch.from_numpy(W["final.norm"]).float() * 0.5)
    assert torch.allclose(model.final_norm.bias, torch.from_numpy(W["final.norm.b"]).float() * 0.5)
    # a layer that borrows its latent ships no matrix for one
    W2 = dict(W)
    W2["l2.mix.dkv"] = W["l0.mix.dkv"]
    d2 = bt.write_model_dir(str(tmp_path / "m2"), bt.B1, W2)
    with pytest.raises(WeightError):
        load_weights(model.weight_specs(), SafetensorsRepo(d2), torch.bfloat16, "cpu", None, log=None)


def test_plain_pieces_by_hand():
    # the norm: deviations over the root of their mean square, then weight and bias
    got = plain.layer_norm(np.array([[1.0, 3.0, 8.0]]), np.array([1.0, 2.0, 1.0]), np.array([0.0, 0.5, 0.0]), 0.0)
    s = math.sqrt((9 + 1 + 16) / 3)
    assert np.allclose(got, [[-3 / s, -2 / s + 0.5, 4 / s]])
    assert np.allclose(plain.rms_norm(np.array([[3.0, 4.0]]), np.array([1.0, 2.0]), 0.0),
                       [[3 / math.sqrt(12.5), 8 / math.sqrt(12.5)]])
    # half-split pairs (i, i + dims/2), the rest passes
    x = np.array([[[1.0, 0.0, 0.0, 2.0, 7.0]]])
    c, s, c2, s2 = math.cos(3.0), math.sin(3.0), math.cos(3.0 * 0.1), math.sin(3.0 * 0.1)
    assert np.allclose(plain.rotate_halves(x, [3], {"dims": 4, "base": 100.0}),
                       [[[c, -2 * s2, s, 2 * c2, 7.0]]])
    # a window of 2 and a sink: the second query sees two keys, the third not the first
    q = np.ones((3, 1, 1))
    k = np.array([1.0, 2.0, 3.0]).reshape(3, 1, 1)
    v = np.array([10.0, 20.0, 30.0]).reshape(3, 1, 1)
    got = plain.softmax_attention(q, k, v, 0.5, 2, np.array([0.25]))[:, 0, 0]
    e = [math.exp(0.5), math.exp(1.0), math.exp(1.5), math.exp(0.25)]
    assert np.allclose(got, [10 * e[0] / (e[0] + e[3]), (10 * e[0] + 20 * e[1]) / (e[0] + e[1] + e[3]),
                             (20 * e[1] + 30 * e[2]) / (e[1] + e[2] + e[3])])
    # the convolution's last column meets the current token, zeros before the start
    assert np.allclose(plain.causal_conv(np.array([[1.0], [2.0]]), np.array([[10.0, 1.0]]), np.array([0.5])),
                       [[1.5], [12.5]])
    # one channel, two states: a decay of its own for each
    y = plain.channel_scan(np.array([[2.0], [1.0]]), np.array([[0.5], [1.0]]), np.array([[-1.0, 0.0]]),
                           np.array([[1.0, 3.0], [2.0, 1.0]]), np.array([[1.0, 0.0], [1.0, 1.0]]), np.array([0.25]))
    # S_1 = 0.5 * 2 * (1, 3); y_1 = 1 + 0.5; S_2 = (1 e^-1 + 2, 3 + 1); y_2 = sum + 0.25
    assert np.allclose(y, [[1.5], [math.exp(-1) + 2 + 4 + 0.25]])
    # routing: group 0 holds the largest score, group 1 the larger sum of two; the correction
    # moves the choice and not the weight
    s = np.array([0.9, 0.1, 0.2, 0.6, 0.5, 0.1])
    assert plain.choose_experts(s, np.zeros(6), 2, 1, 1) == [0, 3]
    assert plain.choose_experts(s, np.array([-0.05, 0, -0.1, 0, 0.05, 0]), 2, 2, 1) == [3, 4]
    assert plain.choose_experts(s, np.array([0, 0, 0.1, 0, 0, 0]), 2, 2, 1) == [0, 2]
    assert plain.choose_experts(s, np.array([0, 0, -0.2, 0, 0, 0.0]), 2, 2, 1) == [3, 4]
    # negative choice scores are still chosen inside the open group
    assert plain.choose_experts(s, np.array([0, 0, 0, -2.0, -2.0, -2.0]), 3, 2, 1) == [0, 2, 1]
    assert plain.choose_experts(s, np.array([-3.0, -3, -3, -4, -4, -4]), 3, 2, 1) == [0, 2, 1]
    # groups of one expert: the strength is that expert's score
    assert plain.choose_experts(s, np.zeros(6), 1, 6, 3) == [0]
    W = {"m.router": np.array([[1.0], [-1.0]]), "m.correction": np.array([0.0, 5.0])}
    for e, g in ((0, 1.0), (1, 2.0)):
        W.update({f"m.e{e}.gate": np.array([[g]]), f"m.e{e}.up": np.array([[1.0]]), f"m.e{e}.down": np.array([[1.0]])})
    got = plain.routed(np.array([[2.0]]), W, "m.", {"router": {"experts": 2, "top": 1, "scale": 3.0}})
    assert np.allclose(got, plain.sigmoid(-2.0) * 3.0 * plain.silu(4.0) * 2.0)


# ---------------------------------------------------- the engine's host side on the CPU
@pytest.fixture()
def emulated(monkeypatch):
    emulated_kernels.install(monkeypatch)


def _engine(cfg, W, page_size, max_tokens, slots=4):
    from tgo_b200.engine.step import Engine
    model = bt.bind_model(cfg, W, torch.float32, "cpu")
    return Engine(model, page_size=page_size, max_tokens=max_tokens, num_slots=slots, graphs=False)


def _check(got, cfg, W, requests, tol=3e-4):
    for rid, toks in requests.items():
        want = plain.forward(cfg, W, toks)
        for p in range(len(toks)):
            assert np.abs(got[(rid, p)] - want[p]).max() <= tol * max(1.0, np.abs(want[p]).max()), (rid, p)


@pytest.mark.parametrize("name", ["B1", "B2", "B3", "B4"])
@pytest.mark.parametrize("family", ["whole", "tail", "portions", "mixed"])
def test_engine_host_side_against_plain(emulated, name, family):
    cfg, page = bt.CONFIGS[name]
    W = bt.make_weights(cfg, 3)
    requests = tiny.random_requests(cfg["vocab"], [37, 9, 1, 50, 18, 26], seed=5)
    trace = {"whole": tiny.trace_whole, "tail": lambda r: tiny.trace_tail(r, 6),
             "portions": tiny.trace_portions,
             "mixed": lambda r: tiny.trace_mixed(r, seed=2, max_live=3, tail=5)}[family](requests)
    # a pool for what is live at once, three state slots: pages and slots come back and go out again
    eng = _engine(cfg, W, page, tiny.max_tokens_of(trace, page), slots=3)
    owners = [dict() for _ in eng.cache.groups]
    got = tiny.run_trace_engine(eng, trace, poison=True, owners=owners)
    _check(got, cfg, W, requests)
    if family == "mixed" and eng.cache.groups:
        assert any(len(ids) > 1 for g in owners for ids in g.values())      # a page was reused


def test_a_lent_latent_is_kept_for_its_farthest_reader(emulated):
    """The first layer's own window is 13; the layer that reads its rows through a window of 30
    decides how long pages stay. The borrowing layers own nothing."""
    from tgo_b200.engine.step import StepEntry
    cfg, page = bt.CONFIGS["B1"]
    W = bt.make_weights(cfg, 3)
    eng = _engine(cfg, W, page, 128)
    assert [(g.kind, g.window, g.planes, g.row_shape, g.calls) for g in eng.model.groups] == \
        [("window", 30, 1, (1, 28), [0]), ("full", None, 1, (1, 26), [3])]
    assert eng.model.state_shapes == {1: (72 * 5 + 3 * 72,), 4: (40 * 24 + 40,)}
    eng.admit("a")
    toks = tiny.random_requests(cfg["vocab"], [90], seed=4)["r0"]
    for o in range(0, 90, 10):
        eng.step([StepEntry("a", toks[o:o + 10], [])])
    held = len(eng.cache.requests["a"].held(0))
    assert 30 <= held * page <= 30 + 2 * page and len(eng.cache.requests["a"].held(1)) == 12
    # a full reader keeps everything
    wide = bt.changed(cfg, ("layers", 2, "mixer", "mask"), ...)
    assert bt.bind_model(wide, W, torch.float32, "cpu").groups[0].kind == "full"


def test_a_borrowing_layer_refuses_a_cache_of_its_own(emulated):
    from tgo_b200.config.spec import LayerCall
    from tgo_b200.engine.model import Model
    from tgo_b200.engine.step import Engine, StepEntry
    from tgo_b200.registry import model_spec_from_config
    cfg, page = bt.CONFIGS["B1"]
    spec = model_spec_from_config(cfg)
    spec.run_order[2] = LayerCall(2)
    model = Model(spec, torch.float32, "cpu")
    W = bt.make_weights(cfg, 3)
    model.bind({w.name: torch.from_numpy(W[w.name]).float() for w in model.weight_specs()})
    eng = Engine(model, page_size=page, max_tokens=64, num_slots=1, graphs=False)
    eng.admit("a")
    with pytest.raises(ValueError, match="borrows"):
        eng.step([StepEntry("a", [1, 2, 3], [0])])


def test_a_reused_state_slot_starts_from_zero(emulated):
    from tgo_b200.engine.step import StepEntry
    cfg, page = bt.CONFIGS["B3"]
    W = bt.make_weights(cfg, 4)
    eng = _engine(cfg, W, page, 64, slots=1)
    first, second = [3, 7, 11, 2, 9, 30, 1], [5, 1, 8, 40]
    for rid, toks in (("a", first), ("b", second)):
        eng.admit(rid)
        got = eng.step([StepEntry(rid, toks, list(range(len(toks))))]).numpy()
        want = plain.forward(cfg, W, toks)
        assert np.abs(got - want).max() <= 3e-4 * max(1.0, np.abs(want).max())
        eng.finish(rid)


def test_a_failing_step_leaves_the_state_alone(emulated, monkeypatch):
    from tgo_b200.engine.step import StepEntry
    from tgo_b200.kernels import ops
    cfg, page = bt.CONFIGS["B1"]
    W = bt.make_weights(cfg, 5)
    eng = _engine(cfg, W, page, 64, slots=2)
    toks = [4, 9, 60, 33, 2, 17, 5, 80, 41]
    eng.admit("a")
    eng.step([StepEntry("a", toks[:4], [])])
    good = ops.channel_scan
    calls = []

    def failing(*a, **k):
        calls.append(1)
        good(*a, **k)
        if len(calls) == 2:              # the second scan: the first has moved already
            raise RuntimeError("no")
    monkeypatch.setattr(ops, "channel_scan", failing)
    with pytest.raises(RuntimeError):
        eng.step([StepEntry("a", toks[4:], [])])
    assert len(calls) == 2
    monkeypatch.setattr(ops, "channel_scan", good)
    assert eng.length("a") == 4
    got = eng.step([StepEntry("a", toks[4:], list(range(5)))]).numpy()
    want = plain.forward(cfg, W, toks)[4:]
    assert np.abs(got - want).max() <= 3e-4 * max(1.0, np.abs(want).max())


def test_parallel_block_around_other_parts(emulated, tmp_path):
    """The arrangement with a feed-forward that joins nothing (dense), and with none at all: the
    mixer's result and the feed-forward's both reach the stream; another norm takes the factor
    on the logits."""
    from dataclasses import replace
    from tgo_b200.config.spec import FeedForwardSpec, NormSpec
    from tgo_b200.engine.model import Model
    from tgo_b200.engine.step import Engine, StepEntry
    from tgo_b200.registry import model_spec_from_config
    cfg, page = bt.CONFIGS["B3"]
    spec = model_spec_from_config(cfg)
    dense = FeedForwardSpec("gated_dense", intermediate_size=24,
                            tensors=(("gate", "mlp.shared.gate"), ("up", "mlp.shared.up"), ("down", "mlp.shared.down")))
    spec.layers[0] = replace(spec.layers[0], feed_forward=dense)
    spec.final_norm = NormSpec("rmsnorm", 1e-5)
    W = bt.make_weights(cfg, 6)
    model = Model(spec, torch.float32, "cpu")
    model.bind({w.name: torch.from_numpy(W[w.name]).float() for w in model.weight_specs()})
    eng = Engine(model, page_size=page, max_tokens=64, num_slots=1, graphs=False)
    eng.admit("a")
    toks = [4, 9, 33, 2, 17]
    got = eng.step([StepEntry("a", toks, list(range(5)))]).numpy()
    x = W["embed"][toks]
    h = plain.layer_norm(x, W["l0.norm1"], W["l0.norm1.b"], 1e-5)
    x = x + plain.selective_scan_mixer(h, W, "l0.mix.", cfg["layers"][0]["mixer"]) + \
        plain.gated(h, W, "l0.mlp.shared.")
    h = plain.layer_norm(x, W["l1.norm1"], W["l1.norm1.b"], 1e-5)
    x = x + plain.selective_scan_mixer(h, W, "l1.mix.", cfg["layers"][1]["mixer"])
    want = plain.rms_norm(x, W["final.norm"], 1e-5) @ W["head"].T * cfg["logit_scale"]
    assert np.abs(got - want).max() <= 3e-4 * np.abs(want).max()
