"""Bekunex on the GPU: every new kernel alone against the plain statement of its mechanism (with
inputs made so that a far key, a window's edge, an ignored sink or gate, a lost or foreign state
shows), then the engine against the plain model: whole prompts, decoding, portions down to two
tokens, mixed batches with pages and state slots that come back, first tokens, long decoding, a
long prompt, and greedy generation through the library's entry point, the scheduler and the
command line."""
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import bekunex_tiny as bt
import plain_bekunex as plain
import tiny

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TOL = {torch.float32: 3e-5, torch.bfloat16: 2e-2}


def dev(x, dtype=torch.float32):
    return torch.from_numpy(np.asarray(x, dtype=np.float32)).to(device=DEV, dtype=dtype)


def ints(x):
    return torch.tensor([int(v) for v in x], dtype=torch.int32, device=DEV)


def host(t):
    return t.detach().float().cpu().numpy().astype(np.float64)


def close(got, want, tol, what=""):
    err = np.abs(host(got) - want).max()
    assert err <= tol * max(1.0, np.abs(want).max()), f"{what}: {err}"


# ------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("out", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("delta", [None, torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,d", [(7, 48), (1, 37), (70, 200), (3, 1030), (2, 4100), (2, 17000)])
def test_layer_norm_with_the_add_and_the_row_selection(T, d, delta, out):
    """Rows whose mean is far larger than their spread: a variance taken as the mean square less
    the squared mean would lose most of its digits."""
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(T + d)
    h = (rng.normal(size=(T, d)) + rng.normal(size=(T, 1)) * 60.0).astype(np.float32).astype(np.float64)
    y = bt.bf16_values(rng.normal(size=(T, d)))
    g, b = rng.normal(size=d) + 1.0, rng.normal(size=d)
    x = h + (y if delta is not None else 0.0)
    want = plain.layer_norm(x, g.astype(np.float32), b.astype(np.float32), 1e-5)
    tol = 2e-4 if out == torch.float32 else 1e-2
    hh = dev(h)
    dl = dev(y, delta) if delta is not None else None
    o = torch.empty((T, d), dtype=out, device=DEV)
    rows = [T - 1, 0, T // 2]
    sel = torch.empty((3, d), dtype=out, device=DEV)
    ops.add_layernorm(hh, dl, dev(g), dev(b), 1e-5, sel, ints(rows))      # leaves the stream alone
    close(sel, want[rows], tol, "selected rows")
    close(hh, h, 0.0)
    ops.add_layernorm(hh, dl, dev(g), dev(b), 1e-5, o)
    close(o, want, tol, "all rows")
    close(hh, x, 1e-6, "the stream has moved on")


def _scan_case(c, N, taps, n, rng):
    """Raw channel inputs, gates, raw steps, B and C of one request; its first token is loud."""
    raw = bt.bf16_values(rng.normal(size=(n, c)))
    raw[0] *= 4.0
    return (raw, bt.bf16_values(rng.normal(size=(n, c)) * 1.5), rng.normal(size=(n, c)).astype(np.float32),
            bt.bf16_values(rng.normal(size=(n, N))), bt.bf16_values(rng.normal(size=(n, N))))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("c,N,taps", [(72, 5, 4), (40, 1, 1), (33, 16, 2), (130, 20, 3), (24, 64, 5), (10, 90, 4),
                                      (14, 256, 2)])
def test_convolution_and_channel_scan_over_portions(c, N, taps, dtype):
    """Three requests in one batch, cut into portions that end before, on and after the kernel's
    groups of 4 and tiles of 32 or 64 tokens (single tokens among them), their states in slots given
    out of order between rows of NaN; against the plain convolution and scan of the whole
    sequences. Decays from nearly none to nearly all; the loud first token shows a state that is
    lost on the way."""
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(c + N)
    lens = (206, 33, 1)
    cuts = [[31, 1, 1, 2, 4, 64, 65, 33, 5], [1, 5, 1, 26], [1]]
    data = [_scan_case(c, N, taps, n, rng) for n in lens]
    w, bias = rng.normal(size=(c, taps)) * 0.6, rng.normal(size=c) * 0.2
    dt_bias, D = rng.normal(size=c) - 1.0, rng.normal(size=c)
    A = -np.exp(rng.normal(size=(c, N)) * 2.0 - 2.0)
    A[0] = -1e-4                                         # a channel that forgets almost nothing
    floats = c * N + (taps - 1) * c
    state = torch.full((6, floats), float("nan"), dtype=torch.float32, device=DEV)
    slot = [4, 0, 2]
    for s in slot:
        state[s].zero_()
    rnd = bt.bf16_values if dtype == torch.bfloat16 else plain.same
    want = []
    for raw, z, dt, B, C in data:
        u = rnd(plain.silu(plain.causal_conv(raw, w.astype(np.float32), bias.astype(np.float32))))
        y = plain.channel_scan(u, plain.softplus(dt + dt_bias.astype(np.float32)), A, B, C, D.astype(np.float32))
        want.append((u, y * plain.silu(z)))
    a2 = dev(A * math.log2(math.e))
    at = [0, 0, 0]
    for step in range(max(len(x) for x in cuts)):
        live = [r for r in range(3) if step < len(cuts[r])]
        sizes = [cuts[r][step] for r in live]
        T = sum(sizes)
        cat = lambda i: np.concatenate([data[r][i][at[r]:at[r] + m] for r, m in zip(live, sizes)])   # noqa: E731
        xz = dev(np.concatenate([cat(0), cat(1)], 1), dtype)
        rbc = dev(np.concatenate([np.zeros((T, 3)), cat(3), cat(4)], 1), dtype)     # views of wider rows
        q_start, seq = ints(np.cumsum([0] + sizes)), ints(np.repeat(np.arange(len(live)), sizes))
        slots = ints([slot[r] for r in live])
        u = torch.empty((T, c), dtype=dtype, device=DEV)
        ops.causal_conv_act(xz[:, :c], dev(w), dev(bias), u, len(live), seq, q_start, slots, state, c * N, keep=False)
        y = torch.empty((T, c), dtype=dtype, device=DEV)
        ops.channel_scan(u, xz[:, c:], dev(cat(2)), dev(dt_bias), a2, rbc[:, 3:3 + N], rbc[:, 3 + N:], dev(D), y,
                         len(live), q_start, slots, state, 0, xz[:, :c], taps, c * N)
        o = 0
        for r, m in zip(live, sizes):
            u_want, y_want = want[r][0][at[r]:at[r] + m], want[r][1][at[r]:at[r] + m]
            close(u[o:o + m], u_want, 3e-5 if dtype == torch.float32 else 1e-2, "convolution")
            scale = np.abs(want[r][1]).max()
            err = np.abs(host(y[o:o + m]) - y_want).max()
            assert err <= (5e-5 if dtype == torch.float32 else 1.5e-2) * scale, (r, at[r], err)
            o += m
            at[r] += m
    assert at == list(lens)
    assert torch.isnan(state[[1, 3, 5]]).all() and not torch.isnan(state[slot]).any()
    kept = host(state[slot[0], c * N:]).reshape(taps - 1, c)
    assert np.abs(kept - data[0][0][lens[0] - taps + 1:]).max() == 0.0 if taps > 1 else True
    # the loud token is still in the slow channel's last output
    quiet = [x.copy() for x in data[0]]
    quiet[0][0] = 0.0
    u = plain.silu(plain.causal_conv(quiet[0], w, bias))
    y = plain.channel_scan(u, plain.softplus(quiet[2] + dt_bias), A, quiet[3], quiet[4], D) * plain.silu(quiet[1])
    assert np.abs(y[-1, 0] - want[0][1][-1, 0]) > 1e-4


def test_slow_decays_do_not_drift_in_float32():
    """4,000 steps of a state that loses a thousandth each: an exponential that is off by a
    fraction of a unit in the last place the same way every time would show."""
    from tgo_b200.kernels import ops
    n, c, N = 4000, 4, 4
    dt = np.full((n, c), -6.9, dtype=np.float32)           # softplus: about 0.001
    A = -np.array([[0.3, 1.0, 0.05, 0.01]] * c)
    x = np.zeros((n, c))
    x[0] = 1000.0
    x[1:] = 1e-3
    B = C = np.ones((n, N))
    want = plain.channel_scan(x, plain.softplus(dt.astype(np.float64)), A, B, C, np.zeros(c))
    state = torch.zeros((1, c * N), dtype=torch.float32, device=DEV)
    y = torch.empty((n, c), dtype=torch.float32, device=DEV)
    big = torch.full((n, c), 40.0, dtype=torch.float32, device=DEV)          # silu(40) = 40
    ops.channel_scan(dev(x), big, dev(dt), None, dev(A * math.log2(math.e)), dev(B), dev(C), None, y, 1,
                     ints([0, n]), ints([0]), state, 0)
    err = np.abs(host(y) / 40.0 - want) / np.abs(want)
    assert err.max() <= 1e-5, err.max()


def _moe_weights(d, E, ff, rng):
    W = {"r.router": bt.bf16_values(rng.normal(size=(E, d)) * 0.6), "r.correction": rng.normal(size=E) * 0.4}
    for e in range(E):
        W[f"r.e{e}.gate"] = bt.bf16_values(rng.normal(size=(ff, d)) / math.sqrt(d))
        W[f"r.e{e}.up"] = bt.bf16_values(rng.normal(size=(ff, d)) / math.sqrt(d))
        W[f"r.e{e}.down"] = bt.bf16_values(rng.normal(size=(d, ff)) / math.sqrt(ff))
    return W


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,d,E,top,ff,count,keep,scale", [
    (9, 48, 12, 3, 24, 4, 2, 2.5), (1, 40, 4, 1, 32, 4, 2, 1.0), (70, 32, 6, 2, 8, 1, 1, 0.7),
    (150, 192, 64, 4, 16, 8, 3, 1.5), (11, 36, 9, 6, 20, 3, 2, 3.0), (5, 64, 160, 5, 8, 40, 3, 1.2), (4, 40, 78, 3, 8, 39, 34, 1.2),
    (33, 24, 5, 5, 12, 5, 5, 1.0)])
def test_experts_chosen_by_logistic_scores_inside_groups(T, d, E, top, ff, count, keep, scale, dtype):
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(d + E)
    x = bt.bf16_values(rng.normal(size=(T, d)))
    W = _moe_weights(d, E, ff, rng)
    stack = lambda r: dev(np.stack([W[f"r.e{e}.{r}"] for e in range(E)]), dtype)       # noqa: E731
    W["r.correction"] = W["r.correction"].astype(np.float32).astype(np.float64)
    extra, beside = rng.normal(size=(T, d)), bt.bf16_values(rng.normal(size=(T, d)))
    stream = rng.normal(size=(T, d)) * 3.0
    mlp = {"router": {"experts": E, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}
    args = (dev(x, dtype), dev(W["r.router"]), None, stack("gate"), stack("up"), stack("down"), top, "silu")

    def run(corr, **kw):
        return ops.moe_feed_forward(*args, scores="sigmoid", correction=dev(corr), groups=count, keep=keep,
                                    renormalize=False, route_scale=scale, **kw)
    # the correction as drawn; one that makes every choice score negative; one that closes the
    # first group although it holds the largest scores
    low = W["r.correction"] - 4.0
    shut = W["r.correction"] + np.where(np.arange(E) < E // count, -5.0, 0.0)
    for corr in (W["r.correction"], low, shut):
        W2 = dict(W, **{"r.correction": corr.astype(np.float32).astype(np.float64)})
        want = plain.routed(x, W2, "r.", mlp)
        close(run(corr), want, TOL[dtype], "alone")
        close(run(corr, extra=dev(extra)), want + extra, TOL[dtype], "with a shared expert's rows")
        for bd in (torch.float32, torch.bfloat16):
            h = dev(stream)
            assert run(corr, extra=dev(extra), beside=dev(beside, bd), residual=h) is None
            close(h, want + extra + beside + stream, TOL[dtype], "into the stream beside another result")
    if top > 1 and keep < count and keep < 30:               # the groups decide something
        free = dict(mlp, router=dict(mlp["router"], groups={"count": 1, "keep": 1}))
        assert np.abs(plain.routed(x, W, "r.", free) - plain.routed(x, W, "r.", mlp)).max() > 0.01


def test_renormalized_logistic_scores():
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(2)
    T, d, E, top, ff = 13, 40, 10, 4, 16
    x, W = bt.bf16_values(rng.normal(size=(T, d))), _moe_weights(40, 10, 16, rng)
    stack = lambda r: dev(np.stack([W[f"r.e{e}.{r}"] for e in range(E)]))              # noqa: E731
    got = ops.moe_feed_forward(dev(x), dev(W["r.router"]), None, stack("gate"), stack("up"), stack("down"), top,
                               "silu", scores="sigmoid", correction=dev(W["r.correction"]), route_scale=2.0)
    s = plain.sigmoid(x @ W["r.router"].T)
    want = np.zeros((T, d))
    for t in range(T):
        chosen = plain.choose_experts(s[t], W["r.correction"].astype(np.float32), top, 1, 1)
        for e in chosen:
            want[t] += 2.0 * s[t, e] / s[t, chosen].sum() * plain.gated(x[t:t + 1], W, f"r.e{e}.")[0]
    close(got, want, 3e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [1, 9, 40, 70])
@pytest.mark.parametrize("H,K,N", [(3, 12, 20), (5, 7, 11), (8, 24, 72), (2, 600, 16)])
def test_a_product_per_head_times_a_gate(H, K, N, T, dtype):
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(H * K + T)
    x = bt.bf16_values(rng.normal(size=(T, H * K)))
    w = bt.bf16_values(rng.normal(size=(H, N, K)) / math.sqrt(K))
    g = bt.bf16_values(rng.normal(size=(T, H * N)) * 2.0)
    for pad in (8, 5):                                       # the gate is a view of a wider row
        wide = dev(np.concatenate([np.zeros((T, pad)), g], 1), dtype)
        y = torch.empty((T, H * N), dtype=dtype, device=DEV)
        ops.head_linear(dev(x, dtype), K, dev(w, dtype), y, N, wide[:, pad:])
        want = np.einsum("thk,hnk->thn", x.reshape(T, H, K), w).reshape(T, -1) * plain.sigmoid(g)
        close(y, want, TOL[dtype], f"pad {pad}")


def _one_plane_case(H, rank, row, n, loud, rng):
    """Cached rows of one request whose row `loud` stands out for every query; channels past
    `rank` are loud in every row and must not leak into the values."""
    q = rng.normal(size=(n, H, row))
    c = rng.normal(size=(n, row))
    direction = rng.normal(size=row)
    direction /= np.linalg.norm(direction)
    q += 3.0 * direction
    c[:, rank:] *= 3.0
    if loud is not None:
        c[loud] = (6.0 + 1.5 * math.sqrt(row)) * direction
    return bt.bf16_values(q), bt.bf16_values(c)


def _run_one_plane(fn, q, c, H, rank, ps, dtype, positions, window):
    """Queries at `positions` over one request's rows in shuffled pages; pages no query may reach
    through its window, and unheld ones, are NaN."""
    n, row = c.shape
    pages = (n + ps - 1) // ps
    table = list(np.random.default_rng(7).permutation(np.arange(1, pages + 3))[:pages])
    plane = torch.full((pages + 3, 1, ps, row), float("nan"), dtype=dtype, device=DEV)
    first = max(0, min(positions) - window + 1) if window else 0
    for j in range(first // ps * ps, n):
        plane[table[j // ps], 0, j % ps] = dev(c[j], dtype)
    bt_ = torch.zeros((2, pages + 2), dtype=torch.int32, device=DEV)
    bt_[1, :pages] = ints(table)
    out = torch.empty((len(positions), H * rank), dtype=dtype, device=DEV)
    fn(dev(q[positions].reshape(len(positions), -1), dtype), out, plane, bt_, ints([1] * len(positions)),
       ints(positions))
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,rank,row,ps,form", [(3, 28, 28, 8, None), (5, 11, 15, 4, None), (20, 48, 64, 16, "tile"),
                                                (4, 32, 32, 16, "tile"), (72, 120, 120, 16, "tile"),
                                                (16, 512, 512, 16, "wide"), (3, 144, 160, 8, "wide"),
                                                (70, 264, 264, 16, "wide"), (5, 200, 232, 4, "wide")])
def test_window_and_sink_over_latent_rows(H, rank, row, ps, form, dtype):
    """Attention over one cache plane whose rows' first `rank` channels are the values, through
    windows shorter and longer than a key tile, one and none, with and without sinks: a loud row
    just inside and just outside the window of query 100; prompt tiles from the start and from
    the middle, single tokens with their keys in 1, 2 and 5 shares."""
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(H + rank)
    n, bf = 150, torch.bfloat16
    sink = rng.normal(size=H) + 2.0
    scale = 6.0 / (3.0 * (6.0 + 1.5 * math.sqrt(row)))       # the loud row's score is about 6
    if form == "tile":
        assert ops.attention_sink_supports(H, 1, row, rank)
        per = ops.attention_sink_tile_tokens(H)
    elif form == "wide":
        assert ops.attention_sink_wide_supports(H, 1, row, rank) and not ops.attention_sink_supports(H, 1, row, rank)
        per = ops.attention_sink_wide_tile_tokens(H)
    for window, loud in ((33, 100 - 33), (33, 100 - 32), (70, 31), (70, 30), (0, 0), (1, 99), (64, 36)):
        q, c = _one_plane_case(H, rank, row, n, loud, rng)
        k = np.repeat(c[:, None, :], H, 1)
        for sk in (sink, None):
            want = plain.softmax_attention(q, k, k[:, :, :rank], scale, window or None, sk).reshape(n, -1)
            sinks = dev(sk) if sk is not None else None
            what = f"window {window} loud {loud} sink {sk is not None}"

            def generic(qq, out, kc, bt_, seq, pos):
                ops.attention_generic(qq, out, H, 1, row, kc, kc, ps, bt_, seq, pos, scale, window, value_dim=rank,
                                      sinks=sinks, value_row=row)
            picks = [100, 99, 101, 149]
            if sk is not None or form is None:
                close(_run_one_plane(generic, q, c, H, rank, ps, dtype, picks, window), want[picks], TOL[dtype],
                      "generic " + what)
            if form is None or dtype != bf:
                continue

            def launch(qq, out, kc, bt_, seq, pos, *tiles, **kw):
                if form == "tile":
                    ops.attention_sink_tile(qq, out, H, 1, row, rank, kc, kc, ps, bt_, seq, pos, scale, window, sinks,
                                            *tiles, value_row=row, **kw)
                else:
                    ops.attention_sink_wide(qq, out, H, 1, row, rank, kc, ps, bt_, seq, pos, scale, window, sinks,
                                            *tiles, **kw)
            for first, count in ((0, n), (71, 60), (100, 1)):
                t0 = list(range(0, count, per))
                tiles = ints(t0), ints([min(per, count - t) for t in t0])
                some = list(range(first, first + count))
                close(_run_one_plane(lambda *a: launch(*a, *tiles), q, c, H, rank, ps, bf, some, window), want[some],
                      2e-2, f"tiles from {first}, " + what)
            for splits in (1, 2, 5):
                some = [0, 1, 31, 32, 33, 63, 64, 69, 70, 99, 100, 101, 149]
                close(_run_one_plane(lambda *a: launch(*a, n_splits=splits), q, c, H, rank, ps, bf, some, window),
                      want[some], 2e-2, f"single tokens in {splits} shares, " + what)
    # the loud row decides query 100's result inside the window and is not there outside it
    q, c = _one_plane_case(H, rank, row, n, 67, rng)
    k = np.repeat(c[:, None, :], H, 1)
    a, b = (plain.softmax_attention(q, k, k[:, :, :rank], scale, w, sink)[100] for w in (33, 34))
    assert np.abs(a - b).max() > 0.3
    free = plain.softmax_attention(q, k, k[:, :, :rank], scale, 33, None)[100]
    assert np.abs(a - free).max() > 0.01                       # the sink matters


# ------------------------------------------------------------------- the engine, end to end
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (cfg, page) in bt.CONFIGS.items():
        W = bt.make_weights(cfg, 13)
        d = bt.write_model_dir(str(tmp_path_factory.mktemp("bekunex" + name)), cfg, W)
        out[name] = (d, cfg, W, page)
    return out


def spread(d):
    d = d - d.mean()
    return math.sqrt((d * d).mean())


CLOSE = 0.0005        # a choice of experts or groups nearer than this may fall either way in bfloat16


def settled(cfg, W, toks):
    """How many of the first tokens come before the request's first close call."""
    margins = []
    plain.forward(cfg, W, toks, margins=margins)
    return next((p for p, m in enumerate(margins) if m < CLOSE), len(toks))


def bounds(cfg, W, requests, dtype):
    """Plain logits per request, the allowed spread of a difference, and how many positions of
    each request it holds for. float32: rounding, everywhere. bfloat16: three times what rounding
    the activations to bfloat16 does to the plain model's own logits on the same requests (the
    largest over their positions), up to the first token whose experts are a close call (which
    the rounding decides; its state carries the choice on)."""
    want = {rid: plain.forward(cfg, W, toks) for rid, toks in requests.items()}
    if dtype == "float32":
        return want, None, {rid: len(toks) for rid, toks in requests.items()}
    upto = {rid: settled(cfg, W, toks) for rid, toks in requests.items()}
    allowed = 3.0 * max(spread(row - want[rid][p]) for rid, toks in requests.items()
                        for p, row in enumerate(plain.forward(cfg, W, toks, rnd=bt.bf16_values)[:upto[rid]]))
    return want, allowed, upto


def rows_close(got, cfg, W, requests, dtype, wide=1e-4):
    want, allowed, upto = bounds(cfg, W, requests, dtype)
    assert got
    loose = 0
    for (rid, p), row in got.items():
        if p >= upto[rid]:
            loose += 1
            assert np.isfinite(row).all(), (rid, p)
            continue
        err = spread(row.astype(np.float64) - want[rid][p])
        bound = wide * want[rid][p].std() if allowed is None else allowed
        assert err <= bound, (rid, p, err, bound)
    return len(got) - loose


FAMILIES = {"whole": tiny.trace_whole, "tail": lambda r: tiny.trace_tail(r, 12),
            "portions": tiny.trace_portions,
            "mixed": lambda r: tiny.trace_mixed(r, seed=4, max_live=4, tail=9)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("family", list(FAMILIES))
@pytest.mark.parametrize("name", sorted(bt.CONFIGS))
def test_replay_against_plain(models, tmp_path, name, family, dtype):
    d, cfg, W, page = models[name]
    requests = tiny.random_requests(cfg["vocab"], [70, 9, 1, 45, 33, 21], seed=6)
    trace = FAMILIES[family](requests)
    got = tiny.run_trace_program(d, dtype, trace, tmp_path / "out", cfg["vocab"],
                                 extra=["--page-size", str(page), "--max-live", "4"])
    assert len(got) == sum(len(t) for t in requests.values())
    rows_close(got, cfg, W, requests, dtype)


@pytest.mark.parametrize("name", ["B1", "B4", "B5"])
def test_float32_cuts_agree_and_pages_and_slots_come_back(models, name):
    """Every cutting gives the same float32 logits to rounding, with NaN in every page nobody
    holds and three state slots for six requests."""
    import tgo_b200
    d, cfg, W, page = models[name]
    requests = tiny.random_requests(cfg["vocab"], [64, 17, 2, 40, 33, 65], seed=7)
    model = tgo_b200.open(d, dtype="float32")
    base = None
    for family in ("whole", "portions", "mixed"):
        trace = tiny.trace_mixed(requests, seed=1, max_live=3, tail=7) if family == "mixed" \
            else FAMILIES[family](requests)
        eng = model.new_engine(page_size=page, max_tokens=tiny.max_tokens_of(trace, page), num_slots=3)
        owners = [dict() for _ in eng.cache.groups]
        got = tiny.run_trace_engine(eng, trace, poison=True, owners=owners)
        rows_close(got, cfg, W, requests, "float32")
        if base is None:
            base = got
        for key, row in got.items():
            assert np.abs(row - base[key]).max() <= 2e-4 * max(1.0, np.abs(base[key]).max()), key
        if family == "mixed":
            assert any(len(ids) > 1 for g in owners for ids in g.values())


def test_a_batch_gives_each_request_what_it_gets_alone(models):
    """Unequal requests in one step (a long portion, a short one, single tokens) against the
    same requests each in an engine of its own: float32, to rounding."""
    import tgo_b200
    from tgo_b200.engine.step import StepEntry
    d, cfg, W, page = models["B1"]
    model = tgo_b200.open(d, dtype="float32")
    reqs = tiny.random_requests(cfg["vocab"], [41, 6, 19, 2], seed=21)
    heads = {rid: max(1, len(t) - 3) for rid, t in reqs.items()}
    alone = {}
    for rid, toks in reqs.items():
        eng = model.new_engine(page_size=page, max_tokens=64, num_slots=1)
        eng.admit(rid)
        alone[(rid, heads[rid] - 1)] = \
            eng.step([StepEntry(rid, toks[:heads[rid]], [heads[rid] - 1])])[0].float().cpu().numpy()
        for p in range(heads[rid], len(toks)):
            alone[(rid, p)] = eng.step([StepEntry(rid, [toks[p]], [0])])[0].float().cpu().numpy()
    eng = model.new_engine(page_size=page, max_tokens=256, num_slots=4)
    for rid in reqs:
        eng.admit(rid)
    got = {}
    lg = eng.step([StepEntry(rid, reqs[rid][:heads[rid]], [heads[rid] - 1]) for rid in reqs])
    for i, rid in enumerate(reqs):
        got[(rid, heads[rid] - 1)] = lg[i].float().cpu().numpy()
    for r in range(3):
        live = [rid for rid in reqs if heads[rid] + r < len(reqs[rid])]
        if not live:
            break
        lg = eng.step([StepEntry(rid, [reqs[rid][heads[rid] + r]], [0]) for rid in live])
        for i, rid in enumerate(live):
            got[(rid, heads[rid] + r)] = lg[i].float().cpu().numpy()
    assert set(got) == set(alone)
    for key, row in got.items():
        assert np.abs(row - alone[key]).max() <= 2e-4 * max(1.0, np.abs(alone[key]).max()), key
    rows_close(got, cfg, W, reqs, "float32")


@pytest.mark.parametrize("name", ["B1", "B5"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_first_tokens_and_a_long_prompt(models, dtype, name):
    import tgo_b200
    from tgo_b200.engine.step import StepEntry
    d, cfg, W, page = models[name]
    model = tgo_b200.open(d, dtype=dtype)
    toks = tiny.random_requests(cfg["vocab"], [150], seed=13)["r0"]
    eng = model.new_engine(page_size=page, max_tokens=192, num_slots=2)
    eng.admit("a")
    got = {}
    for p, t in enumerate(toks):                       # from an empty cache, one by one (graphs)
        got[("a", p)] = eng.step([StepEntry("a", [t], [0])])[0].float().cpu().numpy()
    rows_close(got, cfg, W, {"a": toks}, dtype)
    # 1100 tokens in one step: the many-row products; then a few decoded
    long = tiny.random_requests(cfg["vocab"], [1106], seed=13)["r0"]
    eng = model.new_engine(page_size=page, max_tokens=1152, num_slots=2)
    eng.admit("b")
    picks = [0, 7, 511, 1023, 1024, 1099]
    lg = eng.step([StepEntry("b", long[:1100], picks)]).float().cpu().numpy()
    rows = {("b", p): lg[i] for i, p in enumerate(picks)}
    for p in range(1100, 1106):
        rows[("b", p)] = eng.step([StepEntry("b", [long[p]], [0])])[0].float().cpu().numpy()
    rows_close(rows, cfg, W, {"b": long}, dtype, wide=2e-4)
    eng.check_kernels()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_equal_portions_replayed_from_a_graph(models, dtype):
    """Portions of 256 tokens of one prompt: from the second on they run as a captured graph
    (the scans' states and the cache advance with every replay)."""
    import tgo_b200
    from tgo_b200.engine.step import StepEntry
    d, cfg, W, page = models["B1"]
    model = tgo_b200.open(d, dtype=dtype)
    toks = tiny.random_requests(cfg["vocab"], [256 * 3 + 5], seed=13)["r0"]
    eng = model.new_engine(page_size=page, max_tokens=832, num_slots=2)
    eng.admit("p")
    got = {}
    for o in range(0, 768, 256):
        lg = eng.step([StepEntry("p", toks[o:o + 256], [0, 255])]).float().cpu().numpy()
        got[("p", o)], got[("p", o + 255)] = lg[0], lg[1]
    assert len(eng._portion_graphs) >= 1
    for p in range(768, len(toks)):
        got[("p", p)] = eng.step([StepEntry("p", [toks[p]], [0])])[0].float().cpu().numpy()
    rows_close(got, cfg, W, {"p": toks}, dtype, wide=2e-4)


def test_greedy_generation_through_entry_point_scheduler_and_command_line(models):
    import tgo_b200
    from tgo_b200.sampling.policy import Policy
    d, cfg, W, page = models["B1"]
    prompts = list(tiny.random_requests(cfg["vocab"], [5, 17, 33, 1, 12], seed=8).values())
    want = [plain.greedy(cfg, W, p, 8) for p in prompts]
    assert len({t for o in want for t in o}) > 4
    model = tgo_b200.open(d, dtype="float32")
    assert model.generate(prompts, Policy(max_tokens=8), slots=3, chunk=16, page_size=page) == want
    # so few pages and slots that requests wait for others' to come back
    assert model.generate(prompts, Policy(max_tokens=8), slots=2, chunk=7, pool_tokens=96,
                          page_size=page) == want
    got = tgo_b200.open(d, dtype="bfloat16").generate(prompts, Policy(max_tokens=8), slots=4,
                                                      page_size=page)
    checked = 0
    for p, o in zip(prompts, got):                       # bfloat16: each pick is near the best
        seq = list(p) + list(o)
        z = plain.forward(cfg, W, seq)
        for at in range(len(p) - 1, min(len(seq) - 1, settled(cfg, W, seq))):
            assert z[at].max() - z[at][seq[at + 1]] <= 0.25 * z[at].std()
            checked += 1
    assert checked >= 8
    tgo = os.path.join(tiny.ROOT, "bin", "tgo")
    r = subprocess.run([sys.executable, tgo, "run", "--prompt", " ".join(map(str, prompts[1])),
                        "--max-tokens", "8", "--precision", "f32", "--context", "64", d],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split()] == want[1]
    r = subprocess.run([sys.executable, tgo, "info", d], capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and "Bekunex" in r.stdout
