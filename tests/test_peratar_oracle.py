"""The plain Peratar implementation against hand-worked values and identities (no GPU)."""
import numpy as np

import peratar_helpers as ph
import peratar_oracle as po


def test_rotation_turns_neighbouring_pairs_and_keeps_the_rest():
    x = np.arange(1.0, 7.0)[None, :]
    y = po.rotate_pairs(x, [3], 100.0, 4)
    for i, f in enumerate([1.0, 0.1]):
        c, s = np.cos(3 * f), np.sin(3 * f)
        u, v = x[0, 2 * i], x[0, 2 * i + 1]
        assert np.allclose(y[0, 2 * i:2 * i + 2], [u * c - v * s, v * c + u * s])
    assert np.array_equal(y[0, 4:], x[0, 4:])
    assert np.array_equal(po.rotate_pairs(x, [0], 100.0, 4), x)


def test_rotated_products_depend_on_the_distance_only():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 8)), rng.standard_normal((1, 8))
    a = po.rotate_pairs(q, [9], 50.0, 8) @ po.rotate_pairs(k, [4], 50.0, 8).T
    b = po.rotate_pairs(q, [105], 50.0, 8) @ po.rotate_pairs(k, [100], 50.0, 8).T
    assert np.allclose(a, b)


def test_xielu_meets_at_zero_with_slope_one_half():
    p, q = 0.3, -0.8
    assert po.xielu(np.array(0.0), p, q) == 0.0
    h = 1e-6
    for s in (h, -h):
        assert abs(float(po.xielu(np.array(s), p, q)) / s - 0.5) < 1e-5
    assert np.isclose(float(po.xielu(np.array(2.0), p, q)), np.log1p(np.exp(p)) * 4 + 1)
    assert np.isclose(float(po.xielu(np.array(-2.0), p, q)), (0.5 + np.log1p(np.exp(q))) * (np.exp(-2) + 1) - 1)


def test_norms():
    x = np.array([[1.0, 2.0, 6.0]])
    assert np.allclose(po.layer_norm(x, np.array([1.0, 2.0, 0.0]), 0.0), [[-2 / np.sqrt(14 / 3), -2 / np.sqrt(14 / 3), 0.0]])
    assert np.allclose(po.rms_norm(x, np.ones(3), 2.0), x / np.sqrt(41 / 3 + 2))


def test_absorbed_scores_equal_expanded_ones():
    """(q . W_uk c) = (W_uk^T q) . c, and the same for values: what lets the cache hold c only."""
    rng = np.random.default_rng(1)
    q, uk, uv, c = rng.standard_normal(5), rng.standard_normal((5, 7)), rng.standard_normal((4, 7)), rng.standard_normal((9, 7))
    p = np.exp(rng.standard_normal(9))
    assert np.allclose((c @ uk.T) @ q, c @ (uk.T @ q))
    assert np.allclose(p @ (c @ uv.T), uv @ (p @ c))


def test_a_causal_prefix_does_not_see_what_follows():
    cfg = ph.CONFIGS["mixed"]
    W = ph.weights(cfg, 3)
    ids = np.random.default_rng(2).integers(0, cfg["vocab"], 20)
    full = po.forward(W, cfg, ids)
    assert np.allclose(po.forward(W, cfg, ids[:11]), full[:11])
    assert np.abs(full).max() <= cfg["logit_softcap"]


def test_greedy_extends_by_the_argmax():
    cfg = ph.CONFIGS["one"]
    W = ph.weights(cfg, 4)
    out = po.greedy(W, cfg, [1, 2, 3], 4)
    assert out[2] == int(np.argmax(po.forward(W, cfg, [1, 2, 3] + out[:2])[-1]))
