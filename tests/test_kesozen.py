"""Kesozen without a GPU: the config reader and its refusals, the declared tensor names, the plain
statement's pieces against values worked out by hand, and the engine's host side (run order with a
loop, cache groups and state rows per pass, packing, portions, mixed batches, reused pages and slots)
with torch stand-ins for the kernels, against the plain statement."""
import math

import numpy as np
import pytest
import torch

import emulated_kernels
import kesozen_tiny as kt
import plain_kesozen as plain
import tiny


def test_reader_builds_the_layers_the_file_lists():
    from tgo_b200.registry import model_spec_from_config
    spec = model_spec_from_config(kt.K1)
    assert spec.architecture == "Kesozen" and not spec.tied_head and len(spec.layers) == 6
    assert {ls.block for ls in spec.layers} == {"sandwich_norm_residual"}
    assert spec.embedding_norm.eps == 1e-2 and spec.embedding_norm_name == "embed.norm"
    assert [(c.layer, c.adds_embedding) for c in spec.run_order] == \
        [(0, False), (1, False), (2, False), (3, False), (1, True), (2, False), (3, False), (1, True), (2, False),
         (3, False), (4, False), (5, False)]
    assert all(c.cache_from is None for c in spec.run_order)
    att = spec.layers[0].mixer
    assert (att.kind, att.num_heads, att.num_kv_heads, att.head_dim, att.value_dim, att.scale) == \
        ("sink_attention", 6, 3, 20, 20, 0.3)
    assert att.values_from_keys and att.sink_score == 0.0 and not att.sink and att.window is None
    assert att.output_gate and att.gate_scope == "head" and att.gate_activation == "sigmoid"
    assert (att.position.kind, att.position.rotary_dim, att.position.theta) == ("rope_half_split", 12, 300.0)
    mem = spec.layers[1].mixer
    assert (mem.kind, mem.num_heads, mem.num_kv_heads, mem.head_dim, mem.value_dim, mem.conv_taps, mem.norm_eps) == \
        ("gated_delta", 4, 2, 12, 24, 4, 1e-2)
    dense, moe = spec.layers[0].feed_forward, spec.layers[1].feed_forward
    assert (dense.kind, dense.intermediate_size, dense.activation) == ("plain_dense", 56, "relu_squared")
    assert (moe.experts, moe.top, moe.intermediate_size, moe.router_groups, moe.router_group_best) == \
        (12, 3, 24, (4, 2), 1)
    assert moe.router_scores == "all" and moe.router_correction and not moe.router_renormalize
    assert not moe.gated and moe.shared is None and moe.router_scale == 1.0 and not moe.router_bias
    assert spec.layers[3].feed_forward is None
    assert spec.layers[5].feed_forward.router_groups == (1, 1)
    # no loop: every layer once; no rotation: positions do not enter; kv_heads and vdim by default
    plain_spec = model_spec_from_config(kt.changed(kt.K1, ("loop",), ...))
    assert [c.layer for c in plain_spec.run_order] == list(range(6))
    assert model_spec_from_config(kt.K4).layers[2].mixer.position is None
    bare = kt.changed(kt.changed(kt.K1, ("layers", 4, "mixer", "kv_heads"), ...), ("layers", 4, "mixer", "vdim"), ...)
    assert model_spec_from_config(bare).layers[4].mixer.num_kv_heads == 2


@pytest.mark.parametrize("path,value,word", [
    (("width",), 0, "width"), (("vocab",), ..., "vocab"), (("norm", "eps"), -1.0, "norm.eps"), (("norm",), ..., "norm"),
    (("layers", 0, "type"), "conv", "layers[0].type"), (("layers", 1, "mixer"), None, "layers[1].mixer"),
    (("layers", 0, "mixer", "heads"), ..., "heads"), (("layers", 0, "mixer", "kv_heads"), 4, "kv_heads"),
    (("layers", 0, "mixer", "vdim"), 16, "vdim"), (("layers", 0, "mixer", "scale"), -1.0, "scale"),
    (("layers", 0, "mixer", "rot", "dims"), 5, "rot.dims"), (("layers", 0, "mixer", "rot", "dims"), 22, "rot.dims"),
    (("layers", 0, "mixer", "rot", "base"), 0.0, "rot.base"),
    (("layers", 1, "mixer", "dim"), 257, "dim"), (("layers", 1, "mixer", "conv"), 65, "conv"),
    (("layers", 1, "mixer", "conv"), ..., "conv"), (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 1, "mixer", "vdim"), 1.5, "vdim"),
    (("layers", 0, "mlp", "kind"), "glu", "mlp.kind"), (("layers", 0, "mlp", "ff"), ..., "mlp.ff"),
    (("layers", 0, "mlp"), 3, "mlp"), (("layers", 1, "mlp", "router"), ..., "mlp.router"),
    (("layers", 1, "mlp", "router", "top"), 13, "router.top"), (("layers", 1, "mlp", "expert", "ff"), 0, "expert.ff"),
    (("layers", 1, "mlp", "router", "groups", "count"), 5, "groups.count"),
    (("layers", 1, "mlp", "router", "groups", "keep"), 5, "groups.keep"),
    (("layers", 2, "mlp", "router", "groups", "keep"), 1, "groups.keep"),
    (("loop", "start"), -1, "loop.start"), (("loop", "start"), 4, "loop.stop"), (("loop", "stop"), 7, "loop.stop"),
    (("loop", "times"), 0, "loop.times"), (("loop",), [0, 1], "loop"), (("layers",), [], "layers"),
])
def test_reader_refuses_by_key(path, value, word):
    from tgo_b200.config.qwen3 import ConfigError
    from tgo_b200.registry import model_spec_from_config
    with pytest.raises(ConfigError) as err:
        model_spec_from_config(kt.changed(kt.K1, path, value))
    assert word in str(err.value)


@pytest.mark.parametrize("name", sorted(kt.CONFIGS))
def test_declared_tensors_are_the_weights_the_tests_make(name):
    from tgo_b200.engine.model import Model
    from tgo_b200.registry import model_spec_from_config
    cfg, _ = kt.CONFIGS[name]
    W = kt.make_weights(cfg, 1)
    model = Model(model_spec_from_config(cfg), torch.float32, "cpu")
    declared = {w.name: tuple(w.shape) for w in model.weight_specs() if not w.optional}
    assert declared == {k: tuple(v.shape) for k, v in W.items()}


def test_a_written_folder_loads(tmp_path):
    from tgo_b200.engine.model import Model
    from tgo_b200.registry import model_spec_from_config
    from tgo_b200.weights.binder import WeightError, load_weights
    from tgo_b200.weights.safetensors import SafetensorsRepo
    W = kt.make_weights(kt.K1, 2)
    d = kt.write_model_dir(str(tmp_path / "m"), kt.K1, W)
    model = Model(model_spec_from_config(kt.K1), torch.bfloat16, "cpu")
    weights = load_weights(model.weight_specs(), SafetensorsRepo(d), torch.bfloat16, "cpu", None, log=None)
    for name in ("embed.norm", "l1.mix.A_log", "l1.mix.dt_bias", "l1.mix.q.conv", "l1.mix.norm", "l1.mlp.correction"):
        assert weights[name].dtype == torch.float32, name
    model.bind(dict(weights))
    # q, k and the gate are one product, padded to whole 16-byte rows; there is no value matrix
    att = model.blocks[0].mixer
    assert att.w_qkv.shape == (6 * 20 + 3 * 20 + 8, 48) and not att.w_qkv[-2:].any()
    assert torch.equal(att.sinks, torch.zeros(6))
    mem = model.blocks[1].mixer
    assert mem.w_in.shape == (2 * 24 + 2 * 96 + 8, 48) and mem.conv.shape == (4, 48 + 96)
    assert torch.allclose(mem.decay, torch.exp(torch.from_numpy(W["l1.mix.A_log"])).float())
    # a layer's value matrix, which the design does not have, is refused
    W2 = dict(W)
    W2["l0.mix.v"] = W["l0.mix.k"]
    d2 = kt.write_model_dir(str(tmp_path / "m2"), kt.K1, W2)
    with pytest.raises(WeightError):
        load_weights(model.weight_specs(), SafetensorsRepo(d2), torch.bfloat16, "cpu", None, log=None)


def test_plain_pieces_by_hand():
    assert np.allclose(plain.rms_norm(np.array([[3.0, 4.0]]), np.array([1.0, 2.0]), 0.5),
                       [[3 / math.sqrt(13.0), 8 / math.sqrt(13.0)]])
    x = np.array([[[1.0, 0.0, 0.0, 2.0, 7.0]]])
    c, s, c2, s2 = math.cos(3.0), math.sin(3.0), math.cos(3.0 * 0.1), math.sin(3.0 * 0.1)
    assert np.allclose(plain.rotate_halves(x, [3], {"dims": 4, "base": 100.0}), [[[c, -2 * s2, s, 2 * c2, 7.0]]])
    # one more in the denominator
    q = np.ones((2, 2, 1))
    k = np.array([1.0, -2.0]).reshape(2, 1, 1)
    v = np.array([10.0, 20.0]).reshape(2, 1, 1)
    got = plain.softmax_plus_one(q, k, v, 0.5)
    a, b = math.exp(0.5), math.exp(-1.0)
    assert np.allclose(got[:, 0, 0], [10 * a / (1 + a), (10 * a + 20 * b) / (1 + a + b)])
    assert np.allclose(got[:, 1], got[:, 0])
    # the values are the keys as they were before the rotation
    W = {"m.q": np.array([[1.0], [0.0]]), "m.k": np.array([[2.0], [1.0]]), "m.g": np.array([[0.3]]), "m.o": np.eye(2)}
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "scale": 1.0, "rot": {"dims": 2, "base": 10.0}}
    got = plain.keys_as_values_attention(np.array([[1.0], [1.0]]), W, "m.", m)
    s0, s1 = 2 * math.cos(1.0) - math.sin(1.0) * -1.0, 2.0       # query at 1 on the keys at 0 and 1
    w = math.exp(s0) + math.exp(s1)
    assert np.allclose(got[1], np.array([2.0, 1.0]) * w / (1 + w) / (1 + math.exp(-0.3)))
    # the convolution's last column meets the current token, zeros before the start
    assert np.allclose(plain.causal_conv(np.array([[1.0], [2.0]]), np.array([[10.0, 1.0]])), [[1.0], [12.0]])
    # the memory: what the key finds is taken off what is written, and the query sees the write
    one = np.ones((2, 1, 1))
    y = plain.delta_memory(one * 2.0, one, np.array([4.0, 10.0]).reshape(2, 1, 1), np.array([[0.5], [0.25]]),
                           np.array([[1.0], [0.5]]))
    # S_1 = 4; shrunk to 1, S_2 = 1 + 0.5 (10 - 1) = 5.5
    assert np.allclose(y[:, 0, 0], [8.0, 11.0])
    # routing: a group counts as its largest choice score
    s = np.array([0.9, 0.1, 0.2, 0.6, 0.5, 0.1])
    assert plain.choose_experts(s, np.zeros(6), 2, 1, 1) == [0, 3]
    assert plain.choose_experts(s, np.zeros(6), 2, 2, 1) == [0, 2]
    assert plain.choose_experts(s, np.array([-0.4, 0, 0, 0, 0, 0.0]), 2, 2, 1) == [3, 4]
    assert plain.choose_experts(s, np.array([-3.0, -3, -3, -4, -4, -4]), 3, 2, 1) == [0, 2, 1]     # all negative
    W = {"m.router": np.array([[1.0], [-1.0]]), "m.correction": np.array([0.0, 5.0])}
    for e in (0, 1):
        W.update({f"m.e{e}.up": np.array([[3.0 - 7.0 * e]]), f"m.e{e}.down": np.array([[2.0]])})
    got = plain.routed(np.array([[2.0], [-1.0]]), W, "m.", {"router": {"experts": 2, "top": 1}})
    assert np.allclose(got, [[0.0], [2.0 * 16.0 * math.e / (math.e + 1 / math.e)]])
    assert plain.run_order({"layers": [0, 0, 0], "loop": {"start": 1, "stop": 2, "times": 3}}) == \
        [(0, False), (1, False), (1, True), (1, True), (2, False)]


# ---------------------------------------------------- the engine's host side on the CPU
@pytest.fixture()
def emulated(monkeypatch):
    emulated_kernels.install(monkeypatch)


def _engine(cfg, W, page_size, max_tokens, slots=4):
    from tgo_b200.engine.step import Engine
    model = kt.bind_model(cfg, W, torch.float32, "cpu")
    return Engine(model, page_size=page_size, max_tokens=max_tokens, num_slots=slots, graphs=False)


def _check(got, cfg, W, requests, tol=5e-4):
    for rid, toks in requests.items():
        want = plain.forward(cfg, W, toks)
        for p in range(len(toks)):
            assert np.abs(got[(rid, p)] - want[p]).max() <= tol * max(1.0, np.abs(want[p]).max()), (rid, p)


@pytest.mark.parametrize("name", ["K1", "K2", "K3", "K4"])
@pytest.mark.parametrize("family", ["whole", "tail", "portions", "mixed"])
def test_engine_host_side_against_plain(emulated, name, family):
    cfg, page = kt.CONFIGS[name]
    W = kt.make_weights(cfg, 3)
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


def test_every_pass_of_a_loop_has_a_cache_or_state_of_its_own():
    cfg, _ = kt.CONFIGS["K1"]
    model = kt.bind_model(cfg, kt.make_weights(cfg, 3), torch.float32, "cpu")
    assert [(g.kind, g.planes, g.row_shape, g.calls) for g in model.groups] == \
        [("full", 2, (3, 20), [0]), ("full", 2, (1, 16), [2, 5, 8]), ("full", 2, (2, 28), [10])]
    assert sorted(model.state_shapes) == [1, 3, 4, 6, 7, 9, 11]
    assert model.state_shapes[1] == model.state_shapes[4] == (4 * 12 * 24 + 3 * (2 * 24 + 96),)


def test_the_embedding_output_joins_ahead_of_every_pass_but_the_first(emulated):
    """A layer whose results are nothing, looped three times: the stream is three times the normed
    embedding; blocks that know no pending norm get the same sum."""
    from tgo_b200.engine.step import StepEntry
    cfg = kt._model(40, 24, 1e-5, (0, 1, 3), [(kt._att(2, 1, 8, 4, 100.0, 0.3), kt._dense(16))])
    W = kt.make_weights(cfg, 3)
    W["l0.norm1b"][:] = 0.0
    W["l0.norm2b"][:] = 0.0
    toks = [3, 7, 30, 1]
    e = plain.rms_norm(W["embed"][toks], W["embed.norm"], 1e-5)
    want = plain.rms_norm(3.0 * e, W["final.norm"], 1e-5) @ W["head"].T
    assert np.allclose(want, plain.forward(cfg, W, toks))
    for takes in (True, False):
        eng = _engine(cfg, W, 16, 64, slots=1)
        eng.model.blocks[0].takes_normed = takes
        eng.admit("a")
        got = eng.step([StepEntry("a", toks, [0, 1, 2, 3])]).numpy()
        assert np.abs(got - want).max() <= 1e-4 * np.abs(want).max()


def test_run_order_that_adds_the_embedding_to_itself_is_refused():
    from tgo_b200.config.spec import LayerCall
    from tgo_b200.registry import model_spec_from_config
    spec = model_spec_from_config(kt.K2)
    spec.run_order[0] = LayerCall(0, adds_embedding=True)
    with pytest.raises(ValueError, match="run_order"):
        spec.validate()


def test_a_reused_state_slot_starts_from_zero(emulated):
    from tgo_b200.engine.step import StepEntry
    cfg, page = kt.CONFIGS["K3"]
    W = kt.make_weights(cfg, 4)
    eng = _engine(cfg, W, page, 64, slots=1)
    for rid, toks in (("a", [3, 7, 11, 2, 9, 30, 1]), ("b", [5, 1, 8, 40])):
        eng.admit(rid)
        got = eng.step([StepEntry(rid, toks, list(range(len(toks))))]).numpy()
        want = plain.forward(cfg, W, toks)
        assert np.abs(got - want).max() <= 5e-4 * max(1.0, np.abs(want).max())
        eng.finish(rid)


def test_a_failing_step_leaves_the_state_alone(emulated, monkeypatch):
    from tgo_b200.engine.step import StepEntry
    from tgo_b200.kernels import ops
    cfg, page = kt.CONFIGS["K1"]
    W = kt.make_weights(cfg, 5)
    eng = _engine(cfg, W, page, 64, slots=2)
    toks = [4, 9, 60, 33, 2, 17, 5, 80, 41]
    eng.admit("a")
    eng.step([StepEntry("a", toks[:4], [])])
    good = ops.delta_scan
    calls = []

    def failing(*a, **k):
        calls.append(1)
        good(*a, **k)
        if len(calls) == 3:              # the second pass of the loop: three memories have moved
            raise RuntimeError("no")
    monkeypatch.setattr(ops, "delta_scan", failing)
    with pytest.raises(RuntimeError):
        eng.step([StepEntry("a", toks[4:], [])])
    assert len(calls) == 3
    monkeypatch.setattr(ops, "delta_scan", good)
    assert eng.length("a") == 4
    got = eng.step([StepEntry("a", toks[4:], list(range(5)))]).numpy()
    want = plain.forward(cfg, W, toks)[4:]
    assert np.abs(got - want).max() <= 5e-4 * max(1.0, np.abs(want).max())


def test_attention_refuses_what_it_does_not_offer_together():
    from dataclasses import replace
    from tgo_b200.parts.attention_sink import SinkAttention
    from tgo_b200.registry import model_spec_from_config
    spec = model_spec_from_config(kt.K1).layers[0].mixer
    for change, word in (({"value_dim": 8}, "values"), ({"sink": True}, "sink"), ({"gate_scope": "channel"}, "gate"),
                         ({"conv_taps": 3}, "convolution"), ({"gate_activation": "silu"}, "gate")):
        with pytest.raises(ValueError, match=word):
            SinkAttention(replace(spec, **change), 48, "l0.", "cpu")
