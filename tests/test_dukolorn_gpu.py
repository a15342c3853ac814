"""The Dukolorn decoder in the engine against the plain statement (tests/plain_dukolorn.py): each mechanism's kernels
alone, then whole models through the step function, the cache manager and the scheduler."""
import numpy as np
import pytest
import torch

import plain_dukolorn as PD
import replay_util as R
from dukolorn_fixtures import CONFIGS, TOL, delta, latent, left, make_requests, model_dir, plain_logits, plain_model, right
from engine_fixtures import make_runner
from test_banelix_gpu import _Alone, _i32, _rel
from test_nuvarax_gpu import _feed, _inputs, _portions_and_reuse, _rebind

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
EPS = 1e-5


def _spec(kind, d, **kw):
    from infero_b200.config.spec import MixerSpec
    return MixerSpec(kind=kind, hidden=d, norm_eps=EPS, weight_suffix="", **kw)


# ---- a norm on a sublayer's result, the embedding's norm -----------------------------------------------------------------
@pytest.mark.parametrize("d", [36, 128, 1000, 2048, 4100])
@pytest.mark.parametrize("partial", [False, True])
def test_a_result_is_normed_and_added_and_x_is_handed_on(d, partial):
    from infero_b200 import kernels as K
    from infero_b200.kernels import layer_ops as L
    g = torch.Generator().manual_seed(d)
    T = 9
    rnd = lambda *s: torch.randn(s, generator=g)                                 # noqa: E731
    x, w, ys, b = rnd(T, d) * 3, 1 + 0.3 * rnd(d), rnd(3, T, d), rnd(d)
    y = ys.double().sum(0) + b.double()
    value = K.Partials(ys.to(DEV), b.to(DEV)) if partial else y.float().to(DEV)
    want = x.double() + PD.unit_rms(y, EPS) * w.double()
    for td, tol in ((torch.float32, 4e-6), (torch.bfloat16, 6e-3), (None, 0)):
        xd = x.to(DEV)
        out = torch.empty(T, d, dtype=td, device=DEV) if td else None
        L.sandwich_norm(xd, K.NormedDelta(value, w.to(DEV), EPS), None, 0.0, out)
        assert _rel(xd, want) < 4e-6 and (out is None or _rel(out, want) < tol)
        if out is not None:
            L.sandwich_norm(xd, None, None, 0.0, out)                             # nothing pending: a copy
            assert torch.equal(out, xd.to(td))


@pytest.mark.parametrize("td", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d", [48, 260, 2048])
def test_the_embedding_is_normed(td, d):
    from infero_b200.kernels import layer_ops as L
    g = torch.Generator().manual_seed(d)
    table, w = torch.randn(31, d, generator=g).to(td), 1 + 0.3 * torch.randn(d, generator=g)
    toks = [3, 30, 0, 7, 7]
    want = PD.unit_rms(table.double()[toks], EPS) * w.double()
    x, h = torch.empty(5, d, device=DEV), torch.empty(5, d, dtype=torch.bfloat16, device=DEV)
    ids = _i32([3, -2, 0, 7, 7])                                                   # the second is still on the device
    L.embed_compose(table.to(DEV), ids, x, 1.0, _i32([9, 30]), None, None, None, _i32(range(5)), _i32([0] * 5), _i32([0]), _i32([5]),
                    _i32([0]), 1, False, norm_w=w.to(DEV), eps=EPS, h=h)
    assert _rel(x, want) < 2e-6 and torch.equal(h, x.bfloat16())


# ---- products through a narrow middle -----------------------------------------------------------------------------------
@pytest.mark.parametrize("T", [1, 7, 33, 130])
@pytest.mark.parametrize("H,K,rank", [(2, 64, 24), (3, 7, 1), (5, 26, 70), (1, 300, 33)])
@pytest.mark.parametrize("wd", [torch.float32, torch.bfloat16])
def test_decays_and_gates_through_a_narrow_middle(T, H, K, rank, wd):
    from infero_b200.kernels import layer_ops as L
    g = torch.Generator().manual_seed(T + rank)
    rows = torch.randn(T, rank + 9, generator=g) * 2
    a, w, b, al = rows[:, 5:5 + rank], torch.randn(H * K, rank, generator=g).to(wd), torch.randn(H * K, generator=g), torch.randn(H, generator=g)
    z = a.double() @ w.double().T
    da, dw = rows.to(DEV)[:, 5:5 + rank], w.to(DEV)
    assert _rel(L.low_rank(da, dw), z) < 2e-6
    want = torch.exp(-torch.exp(al.double()).repeat_interleave(K) * PD.softplus(z + b.double()))
    got = L.low_rank(da, dw, "decay", b.to(DEV), al.to(DEV)).cpu().double()
    assert float((got - want).abs().max()) < 2e-5 and bool((got >= 0).all()) and bool((got <= 1).all())
    for tau in (1.0, 16.0):
        want = torch.sigmoid(z + b.double()) ** (1.0 / tau)
        got = L.low_rank(da, dw, "sigmoid", b.to(DEV), tau=tau).cpu().double()
        assert float((got - want).abs().max()) < 5e-6 and bool((got <= 1).all())
    w2 = torch.randn(2 * H * K + 3, 5, generator=g).to(wd)                          # two products of the same rows in one launch
    one, two = L.low_rank(da, dw, beside=(rows.to(DEV)[:, :5], w2.to(DEV)))
    assert _rel(one, z) < 2e-6 and _rel(two, rows[:, :5].double() @ w2.double().T) < 2e-6


# ---- the two memories ----------------------------------------------------------------------------------------------------
def _delta_alone(H, G, K, V, taps, dtype, rank=20, **kw):
    d = max(64, H * V)
    return _Alone(_spec("channel_delta_memory", d, num_heads=H, num_kv_heads=G, head_dim=K, value_dim=V, conv_taps=taps, low_rank=rank),
                  dtype, **kw)


def _decayed_alone(H, K, V, tau, dtype, rank=20, **kw):
    d = max(64, H * V)
    return _Alone(_spec("decayed_memory", d, num_heads=H, head_dim=K, value_dim=V, decay_tau=tau, low_rank=rank), dtype, **kw)


def _lasting(a, shift=4.0, spread=0.3):
    """Decays of a few hundredths a token, different in every channel, so that a state lasts for hundreds of tokens."""
    for k in a.w:
        if k.endswith("dt_bias"):
            a.w[k] = a.w[k] * 4 - shift
        if k.endswith("a2.b"):
            a.w[k] = a.w[k] * 4 + shift
        if k.endswith(".a2"):
            a.w[k] = a.w[k] * spread
    _rebind(a)


DELTA_SHAPES = [(4, 2, 32, 40, 4), (6, 3, 5, 10, 2), (1, 1, 8, 8, 1), (4, 4, 128, 64, 4), (2, 1, 20, 24, 3), (8, 2, 64, 128, 4), (3, 3, 256, 16, 5),
                (2, 2, 300, 12, 2), (2, 1, 508, 8, 6), (3, 3, 37, 5, 4)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,K,V,taps", DELTA_SHAPES)
def test_the_delta_rule_with_decays_per_channel_in_portions_and_single_tokens(dtype, H, G, K, V, taps):
    a = _delta_alone(H, G, K, V, taps, dtype)
    _lasting(a)
    m, w = delta(H, G, K, V, taps), a.weights()
    _portions_and_reuse(a, lambda h: PD.delta_inner(h, w, "mix", m, EPS), H * V, dtype, 5e-5 if dtype == "float32" else 4e-2)


DECAYED_SHAPES = [(4, 32, 48, 8.0), (3, 7, 9, 1.0), (1, 8, 16, 2.5), (2, 128, 128, 16.0), (5, 18, 3, 30.0), (6, 64, 31, 4.0), (2, 260, 20, 12.0),
                  (1, 500, 8, 3.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,K,V,tau", DECAYED_SHAPES)
def test_gated_linear_attention_in_portions_and_single_tokens(dtype, H, K, V, tau):
    a = _decayed_alone(H, K, V, tau, dtype)
    _lasting(a, 1.0)
    m, w = right(H, K, V, tau), a.weights()
    _portions_and_reuse(a, lambda h: PD.right_inner(h, w, "mix", m, EPS), H * V, dtype, 5e-5 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("shift", [-30.0, 30.0])
@pytest.mark.parametrize("rule", ["delta", "decayed"])
def test_decays_at_their_bounds(rule, shift):
    """Channels that forget everything at every token (products of decays underflow), channels that keep everything, side by
    side in one head."""
    H, K, V = 2, 32, 24
    a = _delta_alone(H, H, K, V, 3, "float32") if rule == "delta" else _decayed_alone(H, K, V, 4.0, "float32")
    for k in a.w:
        if k.endswith(("dt_bias", "a2.b")):
            a.w[k] = torch.where(torch.arange(H * K) % 3 == 0, -shift, shift) + a.w[k]
    _rebind(a)
    h = _inputs(150, a.spec.hidden, "float32", 3)
    m = delta(H, H, K, V, 3) if rule == "delta" else right(H, K, V, 4.0)
    want = (PD.delta_inner if rule == "delta" else PD.right_inner)(h.double(), a.weights(), "mix", m, EPS)
    got = _feed(a, h, 90, (16, 2, 15, 3))
    assert torch.isfinite(got).all() and _rel(got[:, :H * V], want) < 1e-4


@pytest.mark.parametrize("rule", ["delta", "decayed"])
def test_a_state_lasts_for_hundreds_of_tokens(rule):
    """One token writes a large value; it is still read six hundred tokens later, whether the tokens come in one portion
    (beside a short one), in portions of 255 or one by one at the end."""
    n = 700
    h = _inputs(n, 64, "float32", 21, 0.5)
    h[5] *= 10.0
    got, w = {}, None
    for how in ("whole", "portions", "tokens"):
        a = _delta_alone(2, 1, 16, 16, 2, "float32", seed=4) if rule == "delta" else _decayed_alone(2, 16, 16, 8.0, "float32", seed=4)
        _lasting(a, 8.0, 0.1)
        w = a.weights()
        if how == "whole":
            got[how] = a.step([("x", h[:20]), ("r", h)])["r"]
        elif how == "portions":
            got[how] = torch.cat([a.step([("r", h[p:p + 255])])["r"] for p in range(0, n, 255)])
        else:
            got[how] = torch.cat([a.step([("r", h[:n - 80])])["r"]] + [a.step([("r", h[p:p + 1])])["r"] for p in range(n - 80, n)])
    if rule == "delta":
        plain = lambda x: PD.delta_inner(x.double(), w, "mix", delta(2, 1, 16, 16, 2), EPS)      # noqa: E731
    else:
        plain = lambda x: PD.right_inner(x.double(), w, "mix", right(2, 16, 16, 8.0), EPS)       # noqa: E731
    want = plain(h)
    for how in got:
        assert _rel(got[how][:, :32], want) < 3e-4, how
    if rule == "decayed":                               # (the delta rule overwrites what it reads again, by design)
        h2 = h.clone()
        h2[5] = 0.0
        assert _rel(plain(h2)[-1:], want[-1:]) > 0.005


@pytest.mark.parametrize("columns", ["1", "2", "4"])
def test_portions_with_one_two_and_four_columns_a_thread(columns):
    """The scans have all three forms; each in a process of its own, since the choice is read once."""
    import os
    import subprocess
    import sys
    code = ("import sys, torch; sys.path[:0] = %r\n"
            "import test_dukolorn_gpu as t\n"
            "for H, K, V in ((2, 128, 40), (3, 20, 6), (2, 64, 31)):\n"
            "    t.test_the_delta_rule_with_decays_per_channel_in_portions_and_single_tokens('float32', H, H, K, V, 4)\n"
            "    t.test_gated_linear_attention_in_portions_and_single_tokens('float32', H, K, V, 4.0)\n") % ([os.path.join(R.ROOT, "tests"), R.ROOT],)
    proc = subprocess.run([sys.executable, "-c", code], env={**os.environ, "INFERO_MEMORY_COLUMNS": columns}, capture_output=True, text=True,
                          timeout=600)
    assert proc.returncode == 0, proc.stderr


# ---- attention: norms, temperature, soft cap, distance bias, sinks -------------------------------------------------------
def _left_alone(H, G, D, V, scale, bias_max, B, cap, temp, dtype, gain=1.0, **kw):
    d = max(64, H * V)
    a = _Alone(_spec("normed_attention", d, num_heads=H, num_kv_heads=G, head_dim=D, value_dim=V, scale=scale, qk_norm_kind="projection",
                     q_temperature=temp, softcap=cap, distance_buckets=B, distance_max=bias_max, sink_per_head=True, scale_values=True),
               dtype, **kw)
    a.w["l0.mix.rel"] = a.w["l0.mix.rel"] * 6.0
    a.w["l0.mix.sink"] = a.w["l0.mix.sink"] * 6.0
    a.w["l0.mix.q.norm"] = a.w["l0.mix.q.norm"] * gain
    _rebind(a)
    return a


LEFT_SHAPES = [(4, 2, 64, 64, 60, 10, 3.0), (6, 3, 10, 6, 12.5, 24, 1.0), (2, 2, 6, 14, 200, 9, 50.0), (1, 1, 16, 16, 2, 2, 8.0),
               (4, 2, 128, 128, 150, 18, 5.0), (8, 4, 48, 16, 90, 7, 2.0), (8, 1, 64, 64, 40, 16, 10.0), (4, 4, 32, 32, 500, 32, 4.0),
               (16, 2, 64, 64, 100, 12, 20.0), (3, 1, 64, 64, 33, 8, 0.5), (6, 2, 80, 80, 75, 20, 3.0), (20, 1, 32, 32, 64, 16, 6.0),
               (4, 2, 64, 64, 60, 10, 0.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,V,bias_max,B,cap", LEFT_SHAPES)
def test_capped_biased_attention_with_sinks_in_portions_and_single_tokens(dtype, H, G, D, V, bias_max, B, cap):
    scale, temp = D ** -0.5, (0.4, 24)
    a = _left_alone(H, G, D, V, scale, bias_max, B, cap, temp, dtype, gain=2.0, pages=128)
    m, w = left(H, G, D, V, scale, bias_max, cap, temp), a.weights()
    d = a.spec.hidden
    h1, h2 = _inputs(330, d, dtype, 7), _inputs(50, d, dtype, 8)
    first = a.step([("a", h1[:63]), ("b", h2[:2])])
    second = a.step([("b", h2[2:50]), ("a", h1[63:64])])
    outs, at = [first["a"], second["a"]], 64
    for size in (2, 1, 1, 62, 65, 1, 70, 17):
        outs.append(a.step([("a", h1[at:at + size])])["a"])
        at += size
    a.close("b")
    third = []
    for i in range(330 - at):                                             # single tokens of two requests side by side
        got = a.step([("a", h1[at + i:at + i + 1])] + ([("c", h2[i:i + 1])] if i < 40 else []))
        outs.append(got["a"])
        if i < 40:
            third.append(got["c"])
    tol = 3e-5 if dtype == "float32" else 4e-2
    assert _rel(torch.cat(outs)[:, :H * V], PD.left_inner(h1.double(), w, "mix", m, EPS)) < tol
    assert _rel(torch.cat([first["b"], second["b"]])[:, :H * V], PD.left_inner(h2.double(), w, "mix", m, EPS)) < tol
    assert _rel(torch.cat(third)[:, :H * V], PD.left_inner(h2[:len(third)].double(), w, "mix", m, EPS)) < tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D,sink", [(64, -40.0), (64, 0.0), (64, 3.0), (40, 3.0), (48, 3.0), (128, 60.0)])
def test_weights_by_distance_and_sink_alone(dtype, D, sink):
    """Keys of zero: head h's weights are the exponentials of its own column of the table, by the bucket of the distance, over
    their sum plus the exponential of its sink; a sink far below changes nothing, one far above leaves nothing."""
    H, G, bias_max, B, n = 4, 2, 50, 12, 140
    a = _left_alone(H, G, D, D, 1.0, bias_max, B, 4.0, (0.5, 8), dtype)
    a.w["l0.mix.k"] = a.w["l0.mix.k"] * 0
    a.w["l0.mix.sink"] = (torch.arange(H) * 0.5 + sink).to(a.td)
    _rebind(a)
    h = _inputs(n, a.spec.hidden, dtype, 2)
    got = _feed(a, h, 100, (7, 2))[:, :H * D].double()
    w = a.weights()
    v = (h.double() @ w["mix.v"].T).view(n, G, D)
    for i in (0, 1, 5, 6, 49, 50, 51, 99, 100, 139):
        e = torch.exp(torch.stack([w["mix.rel"][PD.distance_bucket(i - j, B, bias_max)] for j in range(i + 1)]))       # [i + 1, H]
        p = e / (e.sum(0) + torch.exp(w["mix.sink"]))
        for head in range(H):
            want = (p[:, head:head + 1] * v[:i + 1, head // (H // G)]).sum(0)
            assert float((got[i, head * D:(head + 1) * D] - want).abs().max()) < (2e-5 if dtype == "float32" else 3e-2) * float(v.abs().max()), (i, head)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("back", [0, 1, 15, 16, 17, 255, 256, 257, 300])
@pytest.mark.parametrize("D", [64, 40])
def test_a_far_key_is_found_at_every_distance(dtype, back, D):
    """The key that carries the weight sits at page borders and hundreds of tokens back; in a portion and in single tokens."""
    H, G, V, bias_max, B, scale, cap, temp = 2, 1, D, 64, 8, 0.3, 12.0, (0.3, 100)
    a = _left_alone(H, G, D, V, scale, bias_max, B, cap, temp, dtype, seed=back, pages=64)
    d = a.spec.hidden
    # a token's query is its key as projected from the input with its second half negated: where the last token's input is
    # an earlier one's with that half negated, its query is that token's key and its own key points elsewhere
    a.w["l0.mix.q"] = torch.cat([a.w["l0.mix.k"]] * H)
    a.w["l0.mix.q"][:, d // 2:] *= -1
    a.w["l0.mix.rel"] = a.w["l0.mix.rel"] * 0.2
    _rebind(a)
    n = 330
    h = _inputs(n, d, dtype, back)
    h[n - 1] = h[n - 1 - back]
    h[n - 1, d // 2:] *= -1
    m, w = left(H, G, D, V, scale, bias_max, cap, temp), a.weights()
    want = PD.left_inner(h.double(), w, "mix", m, EPS)
    for first in (11, n - 3):
        got = torch.cat([a.step([(first, h[:first])])[first]] +
                        ([a.step([(first, h[first:])])[first]] if first == 11 else [a.step([(first, h[p:p + 1])])[first] for p in range(first, n)]))
        assert _rel(got[:, :H * V], want) < (3e-5 if dtype == "float32" else 4e-2)
        a.close(first)
    if back:
        h2 = h.clone()
        h2[n - 1 - back] = 0.0
        assert _rel(PD.left_inner(h2.double(), w, "mix", m, EPS)[-1:], want[-1:]) > 0.05


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D", [(4, 2, 64), (2, 1, 128), (6, 3, 48)])
def test_single_tokens_behind_long_contexts(dtype, H, G, D):
    """Contexts that the bf16 kernels cut into splits, beside a short one: sinks count once, however many splits there are."""
    scale, cap, temp, n = D ** -0.5, 4.0, (0.3, 200), 1500
    a = _left_alone(H, G, D, D, scale, 300, 16, cap, temp, dtype, gain=2.0, pages=128)
    a.w["l0.mix.sink"] = a.w["l0.mix.sink"] + 6.0                          # (as much as a thousand keys)
    _rebind(a)
    m, w, d = left(H, G, D, D, scale, 300, cap, temp), a.weights(), a.spec.hidden
    h1, h2 = _inputs(n, d, dtype, 1), _inputs(40, d, dtype, 2)
    a.step([("a", h1[:n - 5]), ("b", h2[:35])])
    got = [a.step([("a", h1[n - 5 + i:n - 4 + i]), ("b", h2[35 + i:36 + i])]) for i in range(5)]
    tol = 3e-5 if dtype == "float32" else 3e-2
    assert _rel(torch.cat([x["a"] for x in got])[:, :H * D], PD.left_inner(h1.double(), w, "mix", m, EPS)[-5:]) < tol
    assert _rel(torch.cat([x["b"] for x in got])[:, :H * D], PD.left_inner(h2.double(), w, "mix", m, EPS)[-5:]) < tol


def test_the_temperature_of_queries_far_out():
    """The factor at the positions where it steps, from the kernel that forms it: queries of unit norm times the factor."""
    from infero_b200.kernels import layer_ops as L
    H, D = 2, 8
    for coef, every in ((0.3, 256), (1.5, 7), (0.0, 3), (0.7, 2.5), (-0.1, 1)):
        pos = [0, 1, 2, 5, 6, 7, 13, 254, 255, 256, 511, 512, 4999, 100000]
        T = len(pos)
        proj = torch.randn(T, H * D, generator=torch.Generator().manual_seed(1)).to(DEV)
        q = torch.empty(T, H * D, device=DEV)
        L.qk_prepare(proj, 0, -1, -1, 1, torch.ones(H * D, device=DEV), None, EPS, None, 1.0, _i32(pos), _i32([0] * T), _i32([[0]]), 16, q,
                     None, None, H, 1, D, D, write_cache=False, temperature=(coef, every))
        want = PD.unit_rms(proj.cpu().double(), EPS) * torch.tensor([[PD.query_temperature(p, coef, every)] for p in pos], dtype=torch.float64)
        assert _rel(q, want) < 2e-6, (coef, every)


# ---- latent attention over a window, with sinks -----------------------------------------------------------------------
def _latent_alone(H, D, Rt, V, C, scale, window, dtype, base=500.0, **kw):
    from infero_b200.config.spec import PositionSpec
    d = max(64, H * V)
    pos = PositionSpec("rope_interleaved", base, Rt) if Rt else None
    a = _Alone(_spec("latent_attention", d, num_heads=H, num_kv_heads=1, head_dim=D, rot_dim=Rt, value_dim=V, latent_dim=C, scale=scale,
                     position=pos, window=window, sink_per_head=True), dtype, **kw)
    a.w["l0.mix.sink"] = a.w["l0.mix.sink"] * 6.0
    _rebind(a)
    return a


LATENT_SHAPES = [(4, 32, 16, 24, 64, 39), (3, 6, 4, 5, 10, 7), (1, 8, 2, 8, 8, 1), (8, 64, 32, 32, 128, 100), (5, 24, 8, 40, 40, 4000),
                 (16, 32, 16, 16, 256, 33), (20, 16, 32, 8, 128, 64), (40, 16, 16, 8, 64, 31), (2, 64, 64, 64, 512, 128), (6, 16, 6, 12, 96, 20)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,Rt,V,C,window", LATENT_SHAPES)
def test_latent_attention_over_a_window_in_portions_and_single_tokens(dtype, H, D, Rt, V, C, window):
    scale = 6.0 / (D + Rt)
    a = _latent_alone(H, D, Rt, V, C, scale, window, dtype, pages=64)
    m, w, d = latent(H, D, Rt, V, C, scale, 500.0, window), a.weights(), a.spec.hidden
    h1, h2 = _inputs(260, d, dtype, 7, 0.4), _inputs(50, d, dtype, 8, 0.4)
    first = a.step([("a", h1[:63]), ("b", h2[:2])])
    second = a.step([("b", h2[2:50]), ("a", h1[63:64])])
    outs, at = [first["a"], second["a"]], 64
    for size in (2, 1, 1, 62, 33, 1, 40):
        outs.append(a.step([("a", h1[at:at + size])])["a"])
        at += size
    a.close("b")
    third = []
    for i in range(260 - at):
        got = a.step([("a", h1[at + i:at + i + 1])] + ([("c", h2[i:i + 1])] if i < 40 else []))
        outs.append(got["a"])
        if i < 40:
            third.append(got["c"])
    tol = 3e-5 if dtype == "float32" else 4e-2
    assert _rel(torch.cat(outs)[:, :H * V], PD.latent_inner(h1.double(), w, "mix", m, EPS)) < tol
    assert _rel(torch.cat([first["b"], second["b"]])[:, :H * V], PD.latent_inner(h2.double(), w, "mix", m, EPS)) < tol
    assert _rel(torch.cat(third)[:, :H * V], PD.latent_inner(h2[:len(third)].double(), w, "mix", m, EPS)) < tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("back,window", [(38, 39), (39, 39), (40, 39), (15, 16), (16, 16), (31, 32), (32, 32), (33, 32), (99, 100), (100, 100), (0, 1), (1, 1),
                                         (200, 201), (201, 201)])
@pytest.mark.parametrize("C", [64, 40])
def test_a_key_just_inside_and_just_outside_the_window(dtype, back, window, C):
    """A key that would take most of the weight, at the window's edge and just beyond it, for a query in a portion and for one
    that comes alone."""
    H, D, Rt, V, scale, n = 2, 16, 16, 32, 2.0, 240
    a = _latent_alone(H, D, Rt, V, C, scale, window, dtype, seed=back, pages=64)
    d = a.spec.hidden
    # the queries' plain parts are made as the keys are, from the input with its second half negated; their rotated parts are 0
    down = a.w["l0.mix.dkv"][:C].float() * a.w["l0.mix.dkv.norm"].float().unsqueeze(1)
    rows = []
    for head in range(H):
        rows += [a.w["l0.mix.uk"][head * D:(head + 1) * D].float() @ down, torch.zeros(Rt, d)]
    q = torch.cat(rows) * 0.3
    q[:, d // 2:] *= -1
    a.w["l0.mix.q"] = q.to(a.td)
    _rebind(a)
    h = _inputs(n, d, dtype, back + 1, 0.5)
    h[n - 1] = h[n - 1 - back]
    h[n - 1, d // 2:] *= -1
    m, w = latent(H, D, Rt, V, C, scale, 500.0, window), a.weights()
    want = PD.latent_inner(h.double(), w, "mix", m, EPS)
    for first in (11, n - 3, n - 1):
        got = [a.step([(first, h[:first])])[first]]
        got += [a.step([(first, h[first:])])[first]] if first == 11 else [a.step([(first, h[p:p + 1])])[first] for p in range(first, n)]
        assert _rel(torch.cat(got)[-4:, :H * V], want[-4:]) < (3e-5 if dtype == "float32" else 4e-2), first
        a.close(first)
    if back:
        h2 = h.clone()
        h2[n - 1 - back] = 0.0
        moved = _rel(PD.latent_inner(h2.double(), w, "mix", m, EPS)[-1:], want[-1:])
        assert moved > 0.05 if back < window else moved == 0.0
        other = PD.latent_inner(h.double(), w, "mix", latent(H, D, Rt, V, C, scale, 500.0, window + (1 if back >= window else -1)), EPS)
        if back in (window - 1, window):
            assert _rel(other[-1:], want[-1:]) > 0.05                     # a window one off would show


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_single_tokens_of_long_contexts_in_ranges(dtype):
    """Contexts cut into ranges of keys, windows that start in the middle of a tile, beside a request shorter than the window;
    sinks count once."""
    from infero_b200.kernels import latent_mma
    H, D, Rt, V, C, scale, window, n = 4, 32, 16, 16, 128, 0.3, 500, 900
    a = _latent_alone(H, D, Rt, V, C, scale, window, dtype, pages=128)
    m, w, d = latent(H, D, Rt, V, C, scale, 500.0, window), a.weights(), a.spec.hidden
    h1, h2 = _inputs(n, d, dtype, 1, 0.4), _inputs(90, d, dtype, 2, 0.4)
    a.step([("a", h1[:n - 6]), ("b", h2[:84])])
    before = latent_mma.launches["cut"]
    got = [a.step([("a", h1[n - 6 + i:n - 5 + i]), ("b", h2[84 + i:85 + i])]) for i in range(6)]
    if dtype == "bfloat16":
        assert latent_mma.launches["cut"] > before
    tol = 3e-5 if dtype == "float32" else 4e-2
    assert _rel(torch.cat([x["a"] for x in got])[:, :H * V], PD.latent_inner(h1.double(), w, "mix", m, EPS)[-6:]) < tol
    assert _rel(torch.cat([x["b"] for x in got])[:, :H * V], PD.latent_inner(h2.double(), w, "mix", m, EPS)[-6:]) < tol


# ---- two mixers side by side, the feed-forward -------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_two_mixers_side_by_side_with_scales(dtype):
    from infero_b200.config.dukolorn import DukolornConfig
    d, H, V, H2, V2 = 160, 4, 16, 2, 24
    cfg = {"vocab": 8, "width": d, "norm": {"eps": EPS}, "layers": [
        {"type": "parallel", "mlp": None, "mixer": {"left": left(H, 2, 16, V, 0.5, 30, 5.0, (0.3, 10)), "right": right(H2, 16, V2, 6.0),
                                                    "left_scale": 0.6, "right_scale": 1.9}}]}
    a = _Alone(DukolornConfig.from_dict(cfg).to_model_spec().blocks[0].mixer, dtype)
    h = _inputs(90, d, dtype, 4)
    m = cfg["layers"][0]["mixer"]
    w = a.weights()
    l = PD.left_inner(h.double(), w, "mix.left", m["left"], EPS)
    r = PD.right_inner(h.double(), w, "mix.right", m["right"], EPS)
    want = torch.cat([0.6 * l, 1.9 * r], dim=1)
    tol = 3e-5 if dtype == "float32" else 4e-2
    got = torch.cat([_feed(a, h, 50, (1, 2, 16))])[:, :H * V + H2 * V2]
    assert _rel(got[:, :H * V], want[:, :H * V]) < tol and _rel(got[:, H * V:], want[:, H * V:]) < tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,ff", [(64, 96), (36, 20), (256, 1024), (2048, 64)])
@pytest.mark.parametrize("T", [1, 8, 40, 257, 600])
def test_the_feed_forward_with_biases(dtype, d, ff, T):
    from infero_b200 import kernels as K
    from infero_b200.config.spec import FeedForwardSpec
    from infero_b200.registry import part_class
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    part = part_class("feed_forward", "swiglu")(FeedForwardSpec(kind="swiglu", hidden=d, intermediate=ff, bias=True, weight_suffix="",
                                                               names=(("gate", "mlp.gate"), ("up", "mlp.up"), ("down", "mlp.down"))), "l0")
    g = torch.Generator().manual_seed(T)
    w = {x.name: (torch.randn(x.shape, generator=g) * (1.0 if x.name.endswith(".b") else x.shape[-1] ** -0.5)).to(td) for x in part.declare()}
    part.bind({k: v.to(DEV) for k, v in w.items()})
    h = _inputs(T, d, dtype, 5)
    y = part.forward(None, h.to(DEV).to(td))
    if isinstance(y, K.Partials):
        y = y.materialize(torch.float32)
    want = PD.biased_swiglu(h.double(), {k[3:]: v.double() for k, v in w.items()}, "mlp")
    assert y.dtype == torch.float32 and _rel(y, want) < (1e-5 if dtype == "float32" else 1.5e-2)


# ---- whole models through the step function ---------------------------------------------------------------------------
def _replay(name, dtype, steps_of, lengths, seed=0, page_size=16, max_seqs=3):
    mdir = model_dir(name)
    reqs = make_requests(name, lengths, seed=seed)
    plain = plain_logits(mdir, reqs)
    steps = steps_of(reqs)
    runner = make_runner(mdir, dtype, R.max_live_tokens(steps, reqs), page_size=page_size, max_seqs=max_seqs)
    got = R.replay_inprocess(runner, steps)
    assert len(got) > 0
    worst, where = R.compare(got, plain)
    each = sorted(R.compare({k: v}, plain)[0] for k, v in got.items())
    most = each[-1 - len(each) // 20]
    print(name, dtype, worst, where, most)
    assert worst <= TOL[dtype][0] and most <= TOL[dtype][1], f"{name} {dtype}: {worst:.3e} at {where}, 95 % of {len(each)} below {most:.3e}"
    assert not runner.manager.requests
    return runner


ALL = [(n, d) for n in sorted(CONFIGS) for d in ("float32", "bfloat16") if (n, d) != ("B", "bfloat16")]   # (B's heads of three numbers
#                                        are normed over themselves: where a read-out is near zero, 16 bits cannot say where it points)


@pytest.mark.parametrize("name,dtype", ALL)
def test_whole_prompts(name, dtype):
    _replay(name, dtype, R.steps_whole, [1, 2, 15, 16, 17, 33, 131])


def test_the_residual_after_every_layer():
    from infero_b200.engine import StepEntry
    from infero_b200.kernels import layer_ops as L
    from infero_b200.parts.block import PostNormBlock
    mdir = model_dir("A")
    toks = make_requests("A", [47], seed=3)["r0"]
    cfg, w = plain_model(mdir)
    trail, seen = [], []
    PD.forward(cfg, w, toks, trail)
    runner = make_runner(mdir, "float32", 64)
    orig = PostNormBlock.forward

    def spy(self, ctx, x, pending, slot):
        out = orig(self, ctx, x, pending, slot)
        after = x.clone()
        L.sandwich_norm(after, out, None, 0.0, None)
        seen.append(after.cpu())
        return out
    PostNormBlock.forward = spy
    try:
        runner.open("a")
        runner.step([StepEntry("a", toks, [len(toks) - 1])])
    finally:
        PostNormBlock.forward = orig
    assert len(seen) == len(trail) == len(cfg["layers"])
    for i, got in enumerate(seen):
        assert _rel(got, trail[i]) < 4e-5, (i, _rel(got, trail[i]))


@pytest.mark.parametrize("name,dtype", ALL)
def test_prompt_then_token_by_token(name, dtype):
    _replay(name, dtype, lambda r: R.steps_tail_decode(r, tail=60), [130, 61, 5])


@pytest.mark.parametrize("name,dtype", ALL)
def test_portions_down_to_two_tokens(name, dtype):
    _replay(name, dtype, lambda r: R.steps_chunked(r, seed=2), [150, 64, 31])
    _replay(name, dtype, lambda r: R.steps_chunked(r, seed=5, sizes=(1, 2, 1, 3, 2, 16, 1, 15, 17)), [70])


@pytest.mark.parametrize("name,dtype", ALL)
def test_mixed_batches_with_slots_and_pages_used_again(name, dtype):
    """Three live requests in exactly three request slots: every later request starts in a slot and on pages that an
    ended one gave back."""
    runner = _replay(name, dtype, lambda r: R.steps_mixed(r, seed=4, max_live=3), [120, 33, 80, 17, 64, 95, 2], max_seqs=3)
    assert runner.manager.pages_reused > 0


def test_a_batch_equals_each_request_alone_bitwise_in_32_bit():
    mdir = model_dir("A")
    reqs = make_requests("A", [50, 21, 37], seed=9)
    together = R.replay_inprocess(make_runner(mdir, "float32", 256, max_seqs=3), [
        {"step": 0, "entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in reqs.items()], "end": list(reqs)}])
    alone = R.replay_inprocess(make_runner(mdir, "float32", 256, max_seqs=3), R.steps_whole(reqs))
    assert together.keys() == alone.keys()
    for k in alone:
        assert np.array_equal(together[k], alone[k]), k


def test_three_hundred_single_tokens():
    _replay("B", "float32", lambda r: R.steps_tail_decode(r, tail=300), [310])
    _replay("D", "bfloat16", lambda r: R.steps_tail_decode(r, tail=300), [305])


def test_long_prompts_in_large_portions():
    """Portions longer than the tiles of the product and attention kernels, cut beside their edges."""
    def steps(reqs):
        (a, ta), (b, tb) = list(reqs.items())[:2]
        return [{"step": 0, "entries": [{"id": a, "tokens": ta[:257], "want": [0, 127, 128, 129, 255, 256]},
                                        {"id": b, "tokens": tb[:40], "want": [39]}], "end": []},
                {"step": 1, "entries": [{"id": b, "tokens": tb[40:425], "want": [0, 87, 88, 384]},
                                        {"id": a, "tokens": ta[257:258], "want": [0]}], "end": []},
                {"step": 2, "entries": [{"id": a, "tokens": ta[258:], "want": list(range(len(ta) - 258))},
                                        {"id": b, "tokens": tb[425:], "want": list(range(len(tb) - 425))}], "end": [a, b]}]
    _replay("D", "bfloat16", steps, [300, 450], max_seqs=2)
    _replay("A", "bfloat16", steps, [300, 450], max_seqs=2)
    _replay("A", "float32", steps, [300, 450], max_seqs=2)


def test_page_size_64():
    _replay("D", "bfloat16", lambda r: R.steps_mixed(r, seed=1, max_live=2), [130, 70, 64], page_size=64)
    _replay("B", "float32", lambda r: R.steps_mixed(r, seed=1, max_live=2), [130, 70, 64], page_size=64)


# ---- the engine's own entry point ------------------------------------------------------------------------------------
def _plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(PD.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_scheduler(name):
    """Several prompts queued at once, more than there are request slots, prompts cut into portions by the
    scheduler's budget, decode steps replayed from captured graphs."""
    from infero_b200.engine import Engine
    from infero_b200.sampling import SamplingParams
    mdir = model_dir(name)
    cfg, w = plain_model(mdir)
    prompts = list(make_requests(name, [19, 40, 3, 27], seed=21).values())
    eng = Engine(mdir, dtype="float32", ctx=128, max_seqs=2, kv_slots=2 * 128, max_batch_tokens=32, cuda_graphs=True)
    params = SamplingParams(temperature=0.0, repetition_penalty=1.0)
    got = eng.generate(prompts, params, max_new_tokens=10, ignore_eos=True)
    for p, g in zip(prompts, got):
        assert g == _plain_greedy(cfg, w, p, 10)
    assert eng.runner.graph_replays > 0


def test_generation_in_bf16_from_captured_graphs_equals_uncaptured_steps():
    from infero_b200.engine import Engine
    from infero_b200.sampling import SamplingParams
    mdir = model_dir("D")
    prompts = list(make_requests("D", [19, 40, 3], seed=22).values())
    params = SamplingParams(temperature=0.0, repetition_penalty=1.0)
    outs = []
    for graphs in (True, False):
        eng = Engine(mdir, dtype="bfloat16", ctx=128, max_seqs=4, kv_slots=4 * 128, max_batch_tokens=64, cuda_graphs=graphs)
        outs.append(eng.generate(prompts, params, max_new_tokens=12, ignore_eos=True))
        if graphs:
            assert eng.runner.graph_replays > 0
    assert outs[0] == outs[1]


def test_the_trace_runner_replays_a_dukolorn_folder(tmp_path):
    mdir = model_dir("A")
    reqs = make_requests("A", [70, 30], seed=2)
    steps = R.steps_mixed(reqs, seed=3, max_live=2)
    got = R.replay_subprocess(mdir, "float32", steps, R.max_live_tokens(steps, reqs), str(tmp_path), CONFIGS["A"]["vocab"])
    worst, where = R.compare(got, plain_logits(mdir, reqs))
    assert worst <= TOL["float32"][0], (worst, where)


def test_the_generate_command_line_on_a_dukolorn_folder():
    import os
    import subprocess
    import sys
    mdir = model_dir("B")
    cfg, w = plain_model(mdir)
    prompt = make_requests("B", [21], seed=8)["r0"]
    exe = os.path.join(R.ROOT, "bin", "generate")
    proc = subprocess.run([sys.executable, exe, mdir] + [str(t) for t in prompt] +
                          ["--greedy", "--repetition-penalty", "1.0", "-n", "7", "--dtype", "float32", "--ignore-eos",
                           "--max-seq-len", "128"], capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr
    lines = proc.stdout.splitlines()
    at = next(i for i, l in enumerate(lines) if l.startswith("kv cache"))
    toks = [int(t) for t in next(l for l in lines[at + 1:] if l.strip()).split()]
    assert toks == _plain_greedy(cfg, w, prompt, 7)
