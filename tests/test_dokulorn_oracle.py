"""The plain Dokulorn implementation against hand-worked values and identities (no GPU)."""
import numpy as np

import dokulorn_helpers as dh
import dokulorn_oracle as do


def test_rotation_turns_entries_half_a_width_apart():
    x = np.arange(1.0, 8.0)[None, :]
    y = do.rotate_halves(x, [3], 100.0, 4)
    for i, f in enumerate([1.0, 0.1]):
        c, s = np.cos(3 * f), np.sin(3 * f)
        u, v = x[0, i], x[0, i + 2]
        assert np.allclose([y[0, i], y[0, i + 2]], [u * c - v * s, v * c + u * s])
    assert np.array_equal(y[0, 4:], x[0, 4:])
    assert np.array_equal(do.rotate_halves(x, [5], 100.0, 0), x)


def test_rotated_products_depend_on_the_distance_only():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 8)), rng.standard_normal((1, 8))
    a = do.rotate_halves(q, [9], 50.0, 8) @ do.rotate_halves(k, [4], 50.0, 8).T
    b = do.rotate_halves(q, [105], 50.0, 8) @ do.rotate_halves(k, [100], 50.0, 8).T
    assert np.allclose(a, b)


def test_norms_and_residual():
    x = np.array([[1.0, 2.0, 2.0]])
    assert np.allclose(do.unit_rms(x, 0.0), x / np.sqrt(3))
    assert np.allclose(do.unit_rms(x, 6.0), x / 3)
    assert np.allclose(do.norm_one_plus(x, np.array([0.0, 1.0, -1.0]), 6.0), [[1 / 3, 4 / 3, 0]])
    assert np.allclose(do.norm_plain(x, np.array([0.0, 1.0, -1.0]), 6.0), [[0, 2 / 3, -2 / 3]])
    assert np.allclose(do.residual(x, -2 * x, np.zeros(3), 3.0, 6.0), x / 3)


def test_a_state_is_the_sum_of_decayed_products():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 4)), rng.standard_normal((9, 4)), rng.standard_normal((9, 3))
    for g in (0.0, 0.7, 1.0):
        o, S = do.decayed_state(q, k, v, g)
        D = np.tril(np.power(g, np.maximum(np.arange(9)[:, None] - np.arange(9), 0).astype(float)))
        assert np.allclose(o, (q @ k.T * D) @ v)
        o1, S1 = do.decayed_state(q[:5], k[:5], v[:5], g)
        o2, S2 = do.decayed_state(q[5:], k[5:], v[5:], g, S1)
        assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)


def test_a_sink_takes_its_share_once():
    s = np.zeros((3, 3))
    assert np.allclose(do.sink_softmax(s, np.log(2.0))[2], np.full(3, 1 / 5))
    assert np.allclose(do.sink_softmax(s, -1e9), np.tril(np.ones((3, 3))) / np.array([[1], [2], [3]]))
    assert np.allclose(do.sink_softmax(np.full((3, 3), 1000.0), 0.0)[0], [1, 0, 0])


def test_soft_cap_and_activations():
    assert np.allclose(do.soft_cap(np.array([-1e3, 0.0, 0.01, 1e3]), 5.0), [-5, 0, 0.01, 5], atol=1e-6)
    assert np.isclose(do.gelu_tanh(1.0), 0.841192) and do.gelu_tanh(0.0) == 0
    assert np.isclose(do.silu(2.0), 2 / (1 + np.exp(-2.0)))


def test_query_heads_share_key_heads_in_runs():
    """Four query heads over two key heads: heads 0, 1 read the first, 2, 3 the second."""
    cfg = dh.config(16, 20, [dh.parallel(dh.attention(4, 2, 8, 4, 4), dh.state(1, 4, 4, (0.9,)))])
    W = {k: v.astype(np.float64) for k, v in dh.weights(cfg, 2).items()}
    W["l0.mix.left.o"] = np.eye(16)
    z = np.random.default_rng(3).standard_normal((6, 16))
    mx = cfg["layers"][0]["mixer"]["left"]
    a = do.grouped_attention(z, W, "l0.mix.left.", mx, 1e-5)
    W["l0.mix.left.v"][4:] = 0
    b = do.grouped_attention(z, W, "l0.mix.left.", mx, 1e-5)
    assert np.array_equal(a[:, :8], b[:, :8]) and not b[:, 8:].any()


def test_a_causal_prefix_does_not_see_what_follows():
    cfg = dh.CONFIGS["mixed"]
    W = dh.weights(cfg, 3)
    ids = np.random.default_rng(2).integers(0, cfg["vocab"], 20)
    assert np.allclose(do.forward(W, cfg, ids[:11]), do.forward(W, cfg, ids)[:11])


def test_greedy_extends_by_the_argmax():
    cfg = dh.CONFIGS["one"]
    W = dh.weights(cfg, 4)
    out = do.greedy(W, cfg, [1, 2, 3], 4)
    assert out[2] == int(np.argmax(do.forward(W, cfg, [1, 2, 3] + out[:2])[-1]))
