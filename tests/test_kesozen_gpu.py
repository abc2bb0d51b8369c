"""Kesozen on the GPU: every new kernel alone against the plain statement of its mechanism (with
inputs made so that a far key, the added one, an ignored gate, a lost or foreign state shows), then
the engine against the plain model: whole prompts, decoding, portions down to two tokens, mixed
batches with pages and state slots that come back, first tokens, long decoding, a long prompt, and
greedy generation through the library's entry point, the scheduler and the command line."""
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import kesozen_tiny as kt
import plain_kesozen as plain
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
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,d", [(7, 48), (1, 37), (40, 200), (3, 1030), (2, 4100)])
def test_embedding_rows_normed_in_the_gather(T, d, dtype):
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(T + d)
    table = kt.bf16_values(rng.normal(size=(23, d)) * 0.02)        # small rows: eps inside the root shows
    g, ids = rng.normal(size=d) + 1.0, rng.integers(0, 23, T)
    want = plain.rms_norm(table[ids] * 1.5, g.astype(np.float32), 1e-3)
    out, copy = torch.empty((T, d), device=DEV), torch.empty((T, d), device=DEV)
    ops.embed_rmsnorm(dev(table, dtype), ints(ids), dev(g), 1e-3, out, copy, 1.5)
    close(out, want, 2e-5)
    assert torch.equal(out, copy)
    ops.embed_rmsnorm(dev(table, dtype), ints(ids), dev(g), 1e-3, copy, None, 1.5)
    assert torch.equal(out, copy)


@pytest.mark.parametrize("out", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,d", [(7, 48), (1, 37), (40, 200), (3, 1030), (5, 2048), (2, 6000), (2, 9000), (2, 1)])
def test_a_result_normed_into_the_stream_and_the_next_norm(T, d, out):
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(T + d)
    f32 = lambda x: x.astype(np.float32).astype(np.float64)                      # noqa: E731
    h, y, e = f32(rng.normal(size=(T, d)) * 3), f32(rng.normal(size=(T, d)) * 0.05), f32(rng.normal(size=(T, d)))
    gy, g = f32(rng.normal(size=d) + 1.0), f32(rng.normal(size=d) + 1.0)
    for extra in (None, e):
        want_h = h + plain.rms_norm(y, gy, 1e-2) + (0.0 if extra is None else extra)
        hh, o = dev(h), torch.empty((T, d), dtype=out, device=DEV)
        ops.norm_add_norm(hh, dev(y), dev(gy), 1e-2, dev(g), 1e-4, o, None if extra is None else dev(extra))
        close(hh, want_h, 1e-5, "the stream")
        close(o, plain.rms_norm(want_h, g, 1e-4), 2e-5 if out == torch.float32 else 1e-2, "the next rows")


def _attention_case(H, G, dim, n, loud, rng):
    """q, k of one request, whose key `loud` stands out for every query; other scores lie around -1,
    so that the added one weighs as much as many keys."""
    q, k = rng.normal(size=(n, H, dim)) * 0.3, rng.normal(size=(n, G, dim)) * 0.3
    direction = rng.normal(size=dim)
    direction /= np.linalg.norm(direction)
    q += 2.0 * direction
    k -= 0.5 * direction
    k[loud] = 4.0 * direction + rng.normal(size=(G, dim)) * 0.3
    return kt.bf16_values(q), kt.bf16_values(k)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dim,rot,ps", [(6, 3, 20, 12, 8), (5, 5, 11, 6, 4), (20, 1, 32, 16, 16), (8, 2, 64, 48, 16),
                                            (6, 2, 112, 112, 8), (3, 1, 200, 64, 16), (9, 3, 24, 0, 16), (1, 1, 8, 2, 16)])
def test_keys_that_are_the_values_with_one_added_and_a_gate_per_head(H, G, dim, rot, ps, dtype):
    """Projection rows (q, k, gate in one row) to the cache and through the attention: prompt tiles
    from the start and from the middle, single tokens with their keys in 1, 2 and 5 shares, the
    generic kernel; a loud key at the start, at page and tile borders and at the newest place."""
    from tgo_b200.kernels import ops
    from tgo_b200.parts.position import RopeHalfSplit
    from tgo_b200.config.spec import PositionSpec
    rng = np.random.default_rng(H * dim)
    n, scale = 150, 0.8
    g = kt.bf16_values(rng.normal(size=(n, H)) * 2.0)
    rnd = kt.bf16_values if dtype == torch.bfloat16 else plain.same
    r = {"dims": rot, "base": 90.0} if rot else None
    table = None
    if rot:
        pos = RopeHalfSplit(PositionSpec("rope_half_split", rotary_dim=rot, theta=90.0), dim, DEV)
    nought = torch.zeros(H, device=DEV)
    tensor_cores = ops.attention_sink_supports(H, G, dim, dim)
    assert tensor_cores == (dim % 8 == 0 and dim <= 128)
    pages = (n + ps - 1) // ps
    moved = [0.0, 0.0]
    for loud in (0, ps - 1, ps, 63, 64, 127, 149):
        q, k = _attention_case(H, G, dim, n, loud, rng)
        qr, kr = (rnd(plain.rotate_halves(z, range(n), r)) for z in (q, k))
        want = plain.softmax_plus_one(qr, kr, k, scale) * plain.sigmoid(g)[:, :, None]
        pad = 8 + -(H * dim + G * dim + H) % 8               # whole 16-byte rows
        rows = np.concatenate([q.reshape(n, -1), k.reshape(n, -1), g, np.full((n, pad), np.nan)], axis=1)
        order = list(np.random.default_rng(loud).permutation(np.arange(1, pages + 3))[:pages])
        kc = torch.full((pages + 3, G, ps, dim), float("nan"), dtype=dtype, device=DEV)
        vc = torch.full_like(kc, float("nan"))
        bt = torch.zeros((2, pages + 2), dtype=torch.int32, device=DEV)
        bt[1, :pages] = ints(order)
        x = dev(rows, dtype)
        slots = ints([order[t // ps] * ps + t % ps for t in range(n)])
        qw, kw = H * dim, G * dim
        kview, gate = x[:, qw:qw + kw], x[:, qw + kw:qw + kw + H]
        if rot:
            table = ops.rope_table(ints(range(n)), pos.inv_freq)
        ops.qkv_bias_rope_cache(x[:, :qw], kview, kview, H, G, dim, dim, None, None, None, table, rot, False, slots,
                                kc, vc, ps)
        close(x[:, qw:qw + kw], k.reshape(n, -1), 0.0, "the projected keys stay as they are")

        def run(fn, picks):
            out = torch.empty((len(picks), H * dim), dtype=dtype, device=DEV)
            i = torch.tensor(picks, device=DEV)
            both = x[i].contiguous()
            fn(both[:, :qw], out, ints([1] * len(picks)), ints(picks), both[:, qw + kw:qw + kw + H])
            return out
        picks = [0, 1, loud, min(loud + 1, 149), 100, 149]
        close(run(lambda qq, o, s, p, gt: ops.attention_generic(qq, o, H, G, dim, kc, vc, ps, bt, s, p, scale, 0,
                                                                sinks=nought, gate=gt), picks),
              want.reshape(n, -1)[picks], TOL[dtype], f"generic, loud {loud}")
        if tensor_cores and dtype == torch.bfloat16:
            per = ops.attention_sink_tile_tokens(H // G)

            def launch(qq, o, s, p, gt, *tiles, **kw):
                ops.attention_sink_tile(qq, o, H, G, dim, dim, kc, vc, ps, bt, s, p, scale, 0, nought, *tiles, gate=gt,
                                        **kw)
            for first, count in ((0, n), (71, 60), (100, 1)):
                t0 = list(range(0, count, per))
                tiles = ints(t0), ints([min(per, count - t) for t in t0])
                some = list(range(first, first + count))
                close(run(lambda *a: launch(*a, *tiles), some), want.reshape(n, -1)[some], 2e-2,
                      f"tiles from {first}, loud {loud}")
            for splits in (1, 2, 5):
                some = [0, 1, 62, 63, 64, 65, 127, 128, 149]
                close(run(lambda *a: launch(*a, n_splits=splits), some), want.reshape(n, -1)[some], 2e-2,
                      f"single tokens in {splits} shares, loud {loud}")
        # the added one and the unrotated values each decide something
        e = np.exp(scale * (qr[:, 0] @ kr[:, 0].T)) * np.tri(n)
        moved[0] = max(moved[0], (1.0 / (1.0 + e.sum(axis=1))).max())
        moved[1] = max(moved[1], np.abs(plain.softmax_plus_one(qr, kr, kr - k, scale)).max())
    assert moved[0] > 0.02 and (moved[1] > 0.2 or not rot)


def _delta_case(H, G, dk, dv, n, rng):
    """Raw projection rows of one request (q, k, v, gate, b, a); its first token is loud."""
    rows = rng.normal(size=(n, 2 * G * dk + 2 * H * dv + 2 * H))
    rows[0] *= 4.0
    return kt.bf16_values(rows)


def _delta_plain(rows, m, conv, dt_bias, a_log, gain, eps):
    """(the rule's results [n, H, dv], the mixer's rows before W_o [n, H dv]) of whole sequences."""
    H, G, dk, dv = m
    n, kw, vw = len(rows), G * dk, H * dv
    x = plain.silu(plain.causal_conv(rows[:, :2 * kw + vw], conv))
    q = np.repeat(plain.unit(x[:, :kw].reshape(n, G, dk)) / math.sqrt(dk), H // G, axis=1)
    k = np.repeat(plain.unit(x[:, kw:2 * kw].reshape(n, G, dk)), H // G, axis=1)
    at = 2 * kw + vw
    decay = np.exp(-np.exp(a_log) * plain.softplus(rows[:, at + vw + H:] + dt_bias))
    o = plain.delta_memory(q, k, x[:, 2 * kw:].reshape(n, H, dv), decay, plain.sigmoid(rows[:, at + vw:at + vw + H]))
    z = plain.silu(rows[:, at:at + vw]).reshape(n, H, dv)
    return o, (plain.rms_norm(o, gain, eps) * z).reshape(n, vw)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,taps", [(4, 2, 12, 24, 4), (1, 1, 1, 4, 1), (3, 1, 9, 7, 9), (2, 2, 32, 16, 2),
                                            (6, 2, 64, 40, 3), (2, 1, 100, 136, 4), (2, 2, 128, 128, 4),
                                            (1, 1, 160, 512, 2), (2, 1, 250, 33, 3), (3, 3, 256, 256, 5), (2, 2, 36, 12, 1)])
def test_delta_rule_over_portions(H, G, dk, dv, taps, dtype):
    """Three requests in one batch, cut into portions that end before, on and after the kernel's pairs
    and tiles of 16 tokens (single tokens among them), their states in slots given out of order
    between rows of NaN; against the plain rule over the whole sequences. Decays from nearly none to
    nearly all; the loud first token shows a memory that is lost on the way."""
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(H * dk + dv)
    lens = (86, 33, 1)
    cuts = [[15, 1, 1, 2, 4, 16, 17, 25, 5], [1, 5, 1, 26], [1]]
    kw, vw = G * dk, H * dv
    C = 2 * kw + vw
    data = [_delta_case(H, G, dk, dv, n, rng) for n in lens]
    f32 = lambda x: x.astype(np.float32).astype(np.float64)                      # noqa: E731
    conv = f32(rng.normal(size=(C, taps)) * 0.6)
    dt_bias, a_log = f32(rng.normal(size=H) - 1.0), f32(rng.normal(size=H) * 1.5 - 1.0)
    dt_bias[0], a_log[0] = -9.0, -2.0                    # a head that forgets almost nothing
    gain, eps = f32(rng.normal(size=dv) + 1.0), 1e-3
    want = [_delta_plain(x, (H, G, dk, dv), conv, dt_bias, a_log, gain, eps) for x in data]
    mem = H * dk * dv
    at_conv = (mem + 3) // 4 * 4
    floats = (at_conv + (taps - 1) * C + 3) // 4 * 4
    state = torch.full((6, floats), float("nan"), dtype=torch.float32, device=DEV)
    slot = [4, 0, 2]
    for s in slot:
        state[s].zero_()
    sizes_ = (H, G, dk, dv)
    takes = ops.delta_step_supports(*sizes_, state, 0)
    assert takes == (dv % 4 == 0 and dk * dv < 50000)
    w, decay, gain_row = dev(conv.T.copy()), dev(np.exp(a_log)), dev(np.tile(gain, H))
    at = [0, 0, 0]
    tol = 5e-5 if dtype == torch.float32 else 1e-2
    for step in range(max(len(x) for x in cuts)):
        live = [r for r in range(3) if step < len(cuts[r])]
        sizes = [cuts[r][step] for r in live]
        T = sum(sizes)
        rows = dev(np.concatenate([data[r][at[r]:at[r] + m] for r, m in zip(live, sizes)]), dtype)
        rows = torch.cat([rows, torch.full((T, (-rows.shape[1]) % 8), float("nan"), dtype=dtype, device=DEV)], dim=1)
        q_start, seq = ints(np.cumsum([0] + sizes)), ints(np.repeat(np.arange(len(live)), sizes))
        slots = ints([slot[r] for r in live])
        raw, z = rows[:, :C], rows[:, C:C + vw]
        b, a = rows[:, C + vw:C + vw + H], rows[:, C + vw + H:C + vw + 2 * H]
        before = state.clone()
        prep = ops.delta_prepare(raw, w, b, a, dev(dt_bias), decay, len(live), *sizes_, seq, q_start, slots, state,
                                 at_conv)
        assert torch.equal(torch.nan_to_num(before), torch.nan_to_num(state))
        y = torch.empty((T, vw), dtype=torch.float32, device=DEV)
        ops.delta_scan(prep, y, len(live), *sizes_, q_start, slots, state, 0, raw, taps, at_conv)
        out = torch.empty((T, vw), dtype=dtype, device=DEV)
        ops.gated_group_norm(y, z, gain_row, out, H, eps, "silu", False)
        if max(sizes) == 1 and takes:
            again, o2 = before, torch.empty_like(out)        # the single-token kernel from the same state
            ops.delta_step(prep, z, dev(gain), eps, o2, len(live), *sizes_, q_start, slots, again, 0, raw, taps, at_conv)
            close(o2, host(out), 1e-4 if dtype == torch.float32 else 1e-2, "single tokens")
            for s in slots.tolist():
                close(again[s], host(state[s]), 1e-6, "the state after single tokens")
            assert torch.isnan(again[[1, 3, 5]]).all()
        o = 0
        for r, m in zip(live, sizes):
            y_want, out_want = (x[at[r]:at[r] + m].reshape(m, -1) for x in want[r])
            scale = np.abs(want[r][0]).max()
            err = np.abs(host(y[o:o + m]) - y_want).max()
            assert err <= tol * scale, (r, at[r], err, scale)
            close(out[o:o + m], out_want, 10 * tol, "normed and gated")
            o += m
            at[r] += m
    assert at == list(lens)
    assert torch.isnan(state[[1, 3, 5]]).all() and not torch.isnan(state[slot]).any()
    if taps > 1:
        kept = host(state[slot[0], at_conv:at_conv + (taps - 1) * C]).reshape(taps - 1, C)
        assert np.abs(kept - data[0][lens[0] - taps + 1:, :C]).max() == 0.0
    if dk > 8:                                           # the loud token is still in the slow head's memory
        quiet = data[0].copy()
        quiet[0] = 0.0
        y = _delta_plain(quiet, (H, G, dk, dv), conv, dt_bias, a_log, gain, eps)[0]
        assert np.abs(y[-1, 0] - want[0][0][-1, 0]).max() > 1e-3 * np.abs(want[0][0][-1, 0]).max()


def test_single_tokens_from_zero_states():
    """A step of single tokens only, many requests, several heads a key head, by its own kernel."""
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(5)
    H, G, dk, dv, taps, B = 6, 3, 48, 72, 4, 37
    C, vw = 2 * G * dk + H * dv, H * dv
    conv, gain = rng.normal(size=(C, taps)).astype(np.float32), (rng.normal(size=dv) + 1).astype(np.float32)
    dt_bias, a_log = np.zeros(H), np.zeros(H)
    data = [_delta_case(H, G, dk, dv, 3, rng) for _ in range(B)]
    at_conv = H * dk * dv
    state = torch.zeros((B + 3, at_conv + (taps - 1) * C), device=DEV)
    slots = ints(np.random.default_rng(1).permutation(B + 3)[:B])
    for t in range(3):
        rows = dev(np.stack([x[t] for x in data]))
        raw, z = rows[:, :C], rows[:, C:C + vw]
        prep = ops.delta_prepare(raw, dev(conv.T.copy()), rows[:, C + vw:C + vw + H], rows[:, C + vw + H:], dev(dt_bias),
                                 dev(np.exp(a_log)), B, H, G, dk, dv, ints(range(B)), ints(range(B + 1)), slots, state,
                                 at_conv)
        out = torch.empty((B, vw), device=DEV)
        ops.delta_step(prep, z, dev(gain), 1e-3, out, B, H, G, dk, dv, ints(range(B + 1)), slots, state, 0, raw, taps,
                       at_conv)
        want = np.stack([_delta_plain(x, (H, G, dk, dv), conv, dt_bias, a_log, gain, 1e-3)[1][t] for x in data])
        close(out, want, 1e-4, f"token {t}")


def test_slow_decays_do_not_drift_in_float32():
    """3,000 steps of a memory that loses a thousandth each and hardly writes: a factor rounded to the
    same side every time would show. Once in one portion, once the last steps one by one."""
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(3)
    n, H, dk, dv = 3000, 2, 8, 4
    rows = np.zeros((n, 2 * H * dk + 2 * H * dv + 2 * H))
    rows[:, :2 * H * dk] = rng.normal(size=(1, 2 * H * dk)) + 3.0 * (rng.random((n, 2 * H * dk)) < 0.01)
    rows[0, 2 * H * dk:2 * H * dk + H * dv] = 50.0
    C, vw = 2 * H * dk + H * dv, H * dv
    rows[:, C + vw:C + vw + H] = -60.0                   # beta: nothing is written
    rows[0, C + vw:C + vw + H] = 60.0                    # but by the first token
    rows[:, C + vw + H:] = 0.0
    rows = kt.bf16_values(rows)
    dt_bias, a_log = np.full(H, -6.9).astype(np.float32), np.array([-0.5, 0.1]).astype(np.float32)
    conv = np.ones((C, 1))
    want = _delta_plain(rows, (H, H, dk, dv), conv, dt_bias.astype(np.float64), a_log.astype(np.float64), np.ones(dv), 1e-6)[0]
    for head in (n, n - 40):
        state = torch.zeros((1, H * dk * dv), device=DEV)
        got = []
        for lo, hi in [(0, head)] + [(t, t + 1) for t in range(head, n)]:
            x = dev(rows[lo:hi])
            prep = ops.delta_prepare(x[:, :C], dev(conv.T.copy()), x[:, C + vw:C + vw + H], x[:, C + vw + H:], dev(dt_bias),
                                     dev(np.exp(a_log.astype(np.float64))), 1, H, H, dk, dv, ints([0] * (hi - lo)),
                                     ints([0, hi - lo]), ints([0]), state, H * dk * dv)
            y = torch.empty((hi - lo, vw), device=DEV)
            ops.delta_scan(prep, y, 1, H, H, dk, dv, ints([0, hi - lo]), ints([0]), state, 0, x[:, :C], 1, H * dk * dv)
            got.append(host(y))
        err = np.abs(np.concatenate(got).reshape(n, H, dv) - want) / np.abs(want).max(axis=(1, 2), keepdims=True)
        assert err.max() <= 2e-5, err.max()


def _moe_weights(d, E, ff, rng):
    W = {"r.router": kt.bf16_values(rng.normal(size=(E, d)) * 0.6), "r.correction": rng.normal(size=E) * 0.1}
    for e in range(E):
        W[f"r.e{e}.up"] = kt.bf16_values(rng.normal(size=(ff, d)) / math.sqrt(d))
        W[f"r.e{e}.down"] = kt.bf16_values(rng.normal(size=(d, ff)) / math.sqrt(ff))
    return W


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,d,E,top,ff,count,keep", [
    (9, 48, 12, 3, 24, 4, 2), (1, 40, 4, 1, 32, 4, 2), (70, 32, 6, 2, 8, 1, 1), (150, 192, 64, 4, 40, 8, 3),
    (11, 36, 9, 6, 20, 3, 2), (5, 64, 160, 5, 8, 40, 3), (4, 40, 78, 3, 8, 39, 34), (33, 24, 5, 5, 12, 5, 5)])
def test_groups_that_count_as_their_largest_choice_score(T, d, E, top, ff, count, keep, dtype):
    from tgo_b200.kernels import ops
    rng = np.random.default_rng(d + E)
    x, W = kt.bf16_values(rng.normal(size=(T, d))), _moe_weights(d, E, ff, rng)
    stack = lambda r: dev(np.stack([W[f"r.e{e}.{r}"] for e in range(E)]), dtype)       # noqa: E731
    mlp = {"router": {"experts": E, "top": top, "groups": {"count": count, "keep": keep}}}
    # the correction as drawn; one that makes every choice score negative; one that closes the first group
    low = W["r.correction"] - 4.0
    shut = W["r.correction"] + np.where(np.arange(E) < E // count, -5.0, 0.0)
    for corr in (W["r.correction"], low, shut):
        corr = corr.astype(np.float32).astype(np.float64)
        want = plain.routed(x, dict(W, **{"r.correction": corr}), "r.", mlp)
        got = ops.moe_feed_forward(dev(x, dtype), dev(W["r.router"]), None, None, stack("up"), stack("down"), top,
                                   "relu_squared", scores="all", correction=dev(corr), groups=count, keep=keep,
                                   renormalize=False, group_best=1)
        close(got, want, TOL[dtype])
    if T > 20 and 1 < E // count and keep < count:           # counting two scores would choose otherwise
        s = plain.softmax(x @ W["r.router"].T) + W["r.correction"]
        runs = np.sort(s.reshape(T, count, -1), axis=2)
        one, two = runs[:, :, -1], runs[:, :, -2:].sum(axis=2)
        assert any(set(np.argsort(-one[t])[:keep]) != set(np.argsort(-two[t])[:keep]) for t in range(T))


# ------------------------------------------------------------------- the engine, end to end
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (cfg, page) in kt.CONFIGS.items():
        W = kt.make_weights(cfg, 13)
        d = kt.write_model_dir(str(tmp_path_factory.mktemp("kesozen" + name)), cfg, W)
        out[name] = (d, cfg, W, page)
    return out


def spread(d):
    d = d - d.mean()
    return math.sqrt((d * d).mean())


CLOSE = 0.005         # a choice of experts or groups nearer than this may fall either way in bfloat16


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
                        for p, row in enumerate(plain.forward(cfg, W, toks, rnd=kt.bf16_values)[:upto[rid]]))
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
@pytest.mark.parametrize("name", sorted(kt.CONFIGS))
def test_replay_against_plain(models, tmp_path, name, family, dtype):
    """K1 through the program that replays traces, the others through the engine it drives."""
    import tgo_b200
    d, cfg, W, page = models[name]
    requests = tiny.random_requests(cfg["vocab"], [70, 9, 1, 45, 33, 21], seed=6)
    trace = FAMILIES[family](requests)
    if name == "K1":
        got = tiny.run_trace_program(d, dtype, trace, tmp_path / "out", cfg["vocab"],
                                     extra=["--page-size", str(page), "--max-live", "4"])
    else:
        eng = tgo_b200.open(d, dtype=dtype).new_engine(
            page_size=page, max_tokens=tiny.max_tokens_of(trace, page), num_slots=4)
        got = tiny.run_trace_engine(eng, trace)
        eng.check_kernels()
    assert len(got) == sum(len(t) for t in requests.values())
    held = rows_close(got, cfg, W, requests, dtype)
    assert held >= len(got) // 2


@pytest.mark.parametrize("name", ["K1", "K4", "K5"])
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
    d, cfg, W, page = models["K1"]
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


@pytest.mark.parametrize("name", ["K1", "K5"])
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
    (the memories and the caches of every pass advance with every replay)."""
    import tgo_b200
    from tgo_b200.engine.step import StepEntry
    d, cfg, W, page = models["K1"]
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
    d, cfg, W, page = models["K1"]
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
    assert r.returncode == 0 and "Kesozen" in r.stdout
