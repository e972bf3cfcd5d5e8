"""Host-side parts of the Tutezen decoder (no GPU): the oracle against second formulations, configuration, weight layout, registry."""
import json

import numpy as np
import pytest

from oracle import tutezen as plain
from skainet_b200 import build, registry
from skainet_b200.tensor import from_bf16_bits
from skainet_b200.tutezen import SsmConfig, TutezenConfig, TutezenDecoder, pad_blocks, pair_rows
from tests import tutezen_models as tm


# ---- the oracle against second formulations ---------------------------------------------------------------
def test_scan_equals_its_sum_and_continues():
    g = np.random.default_rng(0)
    T, H, V, G, N = 9, 4, 3, 2, 5
    x, B, C, dt = g.standard_normal((T, H, V)), g.standard_normal((T, G, N)), g.standard_normal((T, G, N)), g.uniform(0.1, 1, (T, H))
    A, D = g.standard_normal(H), g.standard_normal(H)
    y, S = plain.selective_scan(x, B, C, dt, A, D)
    cum = np.cumsum(-np.exp(A) * dt, axis=0)
    for h in range(H):
        for t in range(T):
            want = D[h] * x[t, h] + sum(np.exp(cum[t, h] - cum[j, h]) * dt[j, h] * (C[t, h // 2] @ B[j, h // 2]) * x[j, h] for j in range(t + 1))
            np.testing.assert_allclose(y[t, h], want, rtol=1e-10, atol=1e-12)
    S4 = plain.selective_scan(x[:4], B[:4], C[:4], dt[:4], A, D)[1]
    y2, S2 = plain.selective_scan(x[4:], B[4:], C[4:], dt[4:], A, D, S4)
    np.testing.assert_allclose(y2, y[4:], rtol=1e-12)
    np.testing.assert_allclose(S2, S, rtol=1e-12)


def test_convolution_looks_back_taps_minus_one():
    u = np.zeros((8, 1))
    u[3] = 1.0
    y = plain.causal_conv(u, np.array([[5.0, 6.0, 7.0]]), np.array([0.5]))
    np.testing.assert_array_equal(y[:, 0], [0.5, 0.5, 0.5, 7.5, 6.5, 5.5, 0.5, 0.5])
    np.testing.assert_array_equal(plain.causal_conv(u, np.array([[2.0]]), np.array([0.0]))[:, 0], 2 * u[:, 0])


def test_adjacent_pairs_turn():
    e = np.zeros((1, 1, 8))
    e[0, 0, 2] = 1.0
    rot = {"dims": 6, "base": 50.0}
    y = plain.rotate_pairs(e, rot, 3)
    a = 3 * 50.0 ** (-2.0 / 6)
    np.testing.assert_allclose(y[0, 0, 2:4], [np.cos(a), np.sin(a)])
    g = np.random.default_rng(1)
    p, q = g.standard_normal((1, 1, 8)), g.standard_normal((1, 1, 8))
    at = lambda v, i: plain.rotate_pairs(v, rot, i)[0, 0]
    assert np.isclose(at(p, 12) @ at(q, 5), at(p, 7) @ at(q, 0))
    np.testing.assert_array_equal(at(p, 9)[6:], p[0, 0, 6:])


def test_window_edges_and_sink():
    assert [j for j in range(20) if plain.window_visible(9, j, 4)] == [6, 7, 8, 9]
    assert [j for j in range(20) if plain.window_visible(2, j, 4)] == [0, 1, 2]
    assert [j for j in range(20) if plain.window_visible(9, j, 1)] == [9]
    s = np.array([0.5, -1.0])
    p = plain.sink_softmax(s, 2.0)
    np.testing.assert_allclose(p, np.exp(s) / (np.exp(s).sum() + np.exp(2.0)))
    np.testing.assert_allclose(plain.sink_softmax(s, -np.inf).sum(), 1.0)


def test_absorbed_queries_meet_latents():
    """Scores and outputs against the latents equal those against expanded keys and values."""
    g = np.random.default_rng(2)
    c, wk, wv, q = g.standard_normal((7, 6)), g.standard_normal((5, 6)), g.standard_normal((4, 6)), g.standard_normal(5)
    s = (c @ wk.T) @ q
    np.testing.assert_allclose(s, c @ (wk.T @ q))
    p = plain.sink_softmax(s, 0.3)
    np.testing.assert_allclose(p @ (c @ wv.T), wv @ (p @ c))


def test_route_takes_the_largest_and_normalises_them():
    e, w = plain.route(np.array([0.1, 3.0, -1.0, 2.0]), 2)
    assert list(e) == [1, 3] and np.isclose(w.sum(), 1.0) and np.isclose(w[0] / w[1], np.e)


def test_loop_order_and_pass_starts():
    cfg = tm.config([tm.ssm()] * 4, loop=(1, 3, 2))
    assert plain.layer_runs(cfg) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert TutezenConfig.from_dict(cfg).runs == [0, 1, 2, 1, 2, 3]


# ---- configuration and weights -------------------------------------------------------------------------------
def test_config_reads_every_size_and_optional_part():
    cfg = TutezenConfig.from_dict(tm.config([tm.ssm(heads=6, groups=3, norm_groups=2, conv=2, mlp=tm.moe(shared=0)), tm.latent(window=0, mlp=tm.dense(9)), tm.latent()],
                                            loop=(0, 2, 3), mult=0.25))
    a, b, c = cfg.layers
    assert (a.mixer.taps, a.mixer.inner, a.mixer.channels, a.ff) == (2, 96, 96 + 2 * 3 * 24, 0)
    assert (a.moe.experts, a.moe.top, a.moe.ff, a.moe.shared_ff) == (6, 2, 24, 0)
    assert (b.mixer.window, b.ff, b.moe, c.mixer.window, c.ff) == (0, 9, None, 17, 0)
    assert cfg.loop == (0, 2, 3) and cfg.residual_mult == 0.25
    s = cfg.tensor_shapes()
    assert s["loop.step"] == (3, 64) and s["l0.mix.in"] == (96 + 96 + 144 + 6, 64) and s["l0.mlp.e5.down"] == (64, 24)
    assert s["l1.mix.uq"] == (3 * 32, 56) and s["l1.mix.dkv"] == (56, 64) and s["l1.mix.o"] == (64, 120) and s["l0.mix.conv"] == (240, 2)
    assert "l0.mlp.shared.up" not in s and "l2.mlp.up" not in s and "l0.norm2" not in s


def test_config_rejects_what_it_does_not_know():
    for change, match in ((lambda c: c["layers"][0].update(type="rwkv"), "unknown mixer"),
                          (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "unknown feed-forward"),
                          (lambda c: c["layers"][0]["mixer"].update(groups=4), "do not divide")):
        bad = tm.config([tm.ssm(mlp=tm.dense())])
        change(bad)
        with pytest.raises(ValueError, match=match):
            TutezenConfig.from_dict(bad)


def test_padded_blocks_and_pairs():
    a = np.arange(12).reshape(6, 2)
    p = pad_blocks(a, 3, 4)
    np.testing.assert_array_equal(p.reshape(2, 4, 2)[:, :3], a.reshape(2, 3, 2))
    assert (p.reshape(2, 4, 2)[:, 3] == 0).all() and pad_blocks(a, 3, 3) is a
    r = pair_rows(a[:3], a[3:])
    assert r.shape == (16, 2)
    np.testing.assert_array_equal(r[:6:2], a[:3])
    np.testing.assert_array_equal(r[1:6:2], a[3:])
    assert not r[6:].any()


def test_joint_rows_give_the_mixers_parts():
    """The padded stack applied to h holds z, x, B, C and dt where the kernels look for them."""
    m = SsmConfig(heads=4, vdim=5, state=6, groups=2, taps=3, norm_groups=1)
    cfg = tm.config([tm.ssm(heads=4, vdim=5, state=6, groups=2, conv=3, norm_groups=1)], width=11)
    bits = tm.weights(cfg, 1)
    get = lambda n: bits[n]
    rows, cols, t, v = TutezenDecoder._ssm(m, "l0.mix.", get, lambda n: from_bf16_bits(bits[n]))
    h = np.random.default_rng(0).standard_normal(11)
    u = from_bf16_bits(np.concatenate(rows)).astype(np.float64) @ h
    raw = from_bf16_bits(bits["l0.mix.in"]).astype(np.float64) @ h
    np.testing.assert_allclose(u[:32].reshape(4, 8)[:, :5].ravel(), raw[:20])                       # z
    np.testing.assert_allclose(u[32:64].reshape(4, 8)[:, :5].ravel(), raw[20:40])                   # x
    np.testing.assert_allclose(u[64:96].reshape(4, 8)[:, :6].ravel(), raw[40:64])                   # B, C: two groups each
    np.testing.assert_allclose(u[96:100], raw[64:68])
    assert len(u) == 104 and not u[100:].any() and v["conv"].shape == (64, 3) and cols[0].shape == (11, 32)


def test_registry_and_family():
    assert registry.architecture_of({"architecture": "Tutezen"}).family == "tutezen"
    part = build.sources("tutezen")
    assert set(part) < set(build.sources()) and not any("lugasun" in f or "llama" in f or "matvec" in f for f in part)


def test_oracle_runs_every_kind_of_layer():
    cfg = tm.config([tm.ssm(mlp=tm.dense()), tm.latent(mlp=tm.moe()), tm.ssm(), tm.latent(mlp=tm.moe(shared=0))], loop=(1, 3, 2))
    w = tm.floats(tm.weights(cfg, 0))
    seen = []
    lg = plain.forward(cfg, w, [1, 2, 3, 4], lambda r, x: seen.append(r))
    assert lg.shape == (4, 90) and np.isfinite(lg).all() and seen == list(range(6))
    np.testing.assert_allclose(plain.forward(json.loads(json.dumps(cfg)), w, [1, 2, 3]), lg[:3], rtol=1e-10, atol=1e-10)
