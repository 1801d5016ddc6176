"""The Dokulorn decoder on the GPU against the plain numpy implementation (oracle/dokulorn_oracle.py).

float32 models are held to rounding in float32, bfloat16 ones to rounding of activations; both are
compared at every layer where the difference would show first."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import dokulorn_helpers as dh
import dokulorn_oracle as do

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 3e-2}   # rms of the difference over rms of the value
SAME = {"float32": 5e-6, "bfloat16": 3e-2}  # the same positions reached by another cut
DT = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def make(pkg, ctx, tmp_path_factory):
    """(config, weights, dtype) -> a loaded model; models and caches are freed with the module."""
    made, caches = [], []

    def build(cfg, W, dtype, max_ctx=512):
        path = dh.write_artifact(tmp_path_factory.mktemp("m"), cfg, W)
        m = pkg.TextModel.load(ctx, path, max_ctx=max_ctx, dtype=pkg.DT_F32 if dtype == "float32" else pkg.DT_BF16)
        made.append(m)
        return m

    def cache(m):
        caches.append(m.make_cache())
        return caches[-1]

    build.cache = cache
    yield build
    for c in caches:
        c.free()
    for m in made:
        m.free()


_ORACLE = {}


def oracle(name, seed, T):
    """Weights, ids, logits and streams of a named configuration, computed once."""
    key = (name, seed, T)
    if key not in _ORACLE:
        cfg = dh.CONFIGS[name]
        W = dh.weights(cfg, seed)
        ids = np.random.default_rng(seed + 1000).integers(0, cfg["vocab"], T)
        _ORACLE[key] = (cfg, W, ids) + do.forward(W, cfg, ids, want_layers=True)
    return _ORACLE[key]


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name,T", [("mixed", 330), ("odd", 140), ("one", 300), ("unrotated", 90), ("wide", 290), ("edges", 100), ("beyond", 60)])
def test_every_layer_and_every_logit(make, name, T, dtype):
    """Rows in one prompt chunk, in windows of 4, and one by one."""
    cfg, W, ids, logits, streams = oracle(name, 7, T)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    for cut in (8192, 4, 1):
        n = T if cut > 1 else min(T, 40)
        c.reset()
        got = m.step_layers(c, ids[:n], prefill_step=cut)
        for i in range(len(cfg["layers"])):
            assert dh.rel(got[i], streams[i, :n]) < TOL[dtype], (cut, "layer", i, dh.rel(got[i], streams[i, :n]))
        c.reset()
        lg = m.step(c, ids[:n], range(n), prefill_step=cut)
        assert dh.rel(lg, logits[:n]) < TOL[dtype], (cut, dh.rel(lg, logits[:n]))


@pytest.mark.parametrize("dtype", DT)
def test_a_prompt_of_many_state_chunks(make, dtype):
    """Long enough that the states are kept and carried many times, cut at, before and after those places."""
    T = 2360
    cfg = dh.config(64, 50, [dh.retention(1, 16, 24, (0.9995,), base=1e6), dh.parallel(dh.attention(2, 1, 16, 16, 8, base=1e6), dh.state(1, 24, 16, (0.998,)))])
    W = dh.weights(cfg, 71)
    ids = np.random.default_rng(72).integers(0, cfg["vocab"], T)
    want = do.forward(W, cfg, ids)
    m = make(cfg, W, dtype, max_ctx=T)
    c = make.cache(m)
    for cut in ((T,), (256, 512, T - 768), (255, 1, 256, T - 512), (2303, T - 2303), (2305, T - 2305)):
        c.reset()
        rows, lo = [], 0
        for n in cut:
            rows.append(m.step(c, ids[lo:lo + n], range(n)))
            lo += n
        got = np.concatenate(rows)
        per_row = np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())
        assert dh.rel(got, want) < TOL[dtype] and per_row.max() < 3 * TOL[dtype], (cut, dh.rel(got, want), int(per_row.argmax()), per_row.max())


# ------------------------------------------------------------------ one mechanism at a time
def silence(cfg, W, keep):
    """Weights under which only the mechanisms in `keep` act: an output matrix or an output norm of zeros removes one."""
    W = {k: v.copy() for k, v in W.items()}
    for i, ly in enumerate(cfg["layers"]):
        p = "l%d." % i
        if ly["type"] == "retention" and "retention" not in keep:
            W[p + "mix.o"][:] = 0
        if ly["type"] == "parallel":
            if "left" not in keep:
                W[p + "mix.left.out"][:] = 0
            if "right" not in keep:
                W[p + "mix.right.out"][:] = 0
        if ly["mlp"] is not None and "ff" not in keep:
            W[p + "mlp.down"][:] = 0
    return W


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("keep", [["retention"], ["left"], ["right"], ["ff"], ["left", "right"], []], ids=lambda k: "+".join(k) or "residual")
def test_one_mechanism_alone(make, keep, dtype):
    cfg = dh.CONFIGS["mixed"]
    W = silence(cfg, dh.weights(cfg, 21), keep)
    ids = np.random.default_rng(5).integers(0, cfg["vocab"], 70)
    want = do.forward(W, cfg, ids, want_layers=True)[1]
    m = make(cfg, W, dtype)
    c = make.cache(m)
    for cut in (8192, 3):
        c.reset()
        got = m.step_layers(c, ids, prefill_step=cut)
        for i in range(len(want)):
            assert dh.rel(got[i], want[i]) < TOL[dtype], (keep, cut, i)


def small(**over):
    """Two layers with everything, whose constants the tests change one at a time."""
    left = dh.attention(4, 2, 16, 8, 8, base=100.0, softcap=20.0)
    right = dh.state(2, 16, 24, (0.9, 0.99))
    ret = dh.retention(2, 16, 24, (0.95, 0.7), rot_dims=8, base=50.0)
    left.update(over.pop("left", {}))
    right.update(over.pop("right", {}))
    ret["mixer"].update(over.pop("ret", {}))
    return dh.config(64, 80, [dh.parallel(left, right, 48), ret], **over)


@pytest.mark.parametrize("change", [dict(eps=0.5), dict(alpha=0.25), dict(alpha=6.0), dict(scale=0.3), dict(left={"scale": 1.5}), dict(left={"scale": -0.5}),
                                    dict(left={"softcap": 0.5}), dict(left={"scale": 1.5, "softcap": 1.0}), dict(left={"rot": dh.rot(16, 100.0)}),
                                    dict(left={"rot": dh.rot(8, 7.0)}), dict(left={"rot": dh.rot(0, 7.0)}), dict(right={"decay": [0.3, 1.0]}),
                                    dict(ret={"decay": [0.2, 1.0]}), dict(ret={"rot": dh.rot(16, 50.0)}), dict(ret={"rot": dh.rot(8, 5.0)})],
                         ids=lambda c: json.dumps(c))
def test_every_constant_is_read(make, change):
    """Each changes the result visibly, and the result follows."""
    W = dh.weights(small(), 41)
    ids = np.arange(40) * 3 % 80
    plain = do.forward(W, small(), ids)
    cfg = small(**json.loads(json.dumps(change)))
    want = do.forward(W, cfg, ids)
    assert dh.rel(want, plain) > 100 * TOL["float32"]
    for dtype in DT:
        m = make(cfg, W, dtype)
        c = make.cache(m)
        for cut in (8192, 1):
            c.reset()
            assert dh.rel(m.step(c, ids, range(40), prefill_step=cut), want) < TOL[dtype], (dtype, cut)


@pytest.mark.parametrize("dtype", DT)
def test_sinks_first_tokens_and_last(make, dtype):
    """Sinks far below, at and far above the scores: from the first token on and behind a long prompt,
    each equal to the plain implementation and unlike the one without sinks."""
    cfg = small(alpha=0.3)
    ids = np.random.default_rng(6).integers(0, 80, 300)
    for value in (-20.0, 0.0, 3.0, 12.0):
        W = silence(cfg, dh.weights(cfg, 42), ["left"])
        W["l0.mix.left.sink"] = dh.bf16_round(np.array([value, value + 1, value - 1, value], np.float32))
        bare = dict(W)
        bare["l0.mix.left.sink"] = np.full(4, -1e4, np.float32)
        want = do.forward(W, cfg, ids)
        if value >= 0:  # the output norm takes a common factor away: unequal sinks stay visible, most of all at the start
            assert dh.rel(do.forward(bare, cfg, ids[:5]), want[:5]) > 3 * TOL[dtype]
        m = make(cfg, W, dtype)
        c = make.cache(m)
        for cut in ((300,), (1,) * 6 + (294,), (4, 290, 1, 1, 4), (70, 230)):
            c.reset()
            rows, lo = [], 0
            for n in cut:
                rows.append(m.step(c, ids[lo:lo + n], range(n)))
                lo += n
            got = np.concatenate(rows)
            per_row = np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())
            assert per_row.max() < 3 * TOL[dtype], (value, cut, int(per_row.argmax()), per_row.max())


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("group,dim", [(24, 24), (130, 130), (520, 520), (700, 700), (5, 5)])
def test_head_norms_of_every_width(make, group, dim, dtype):
    """Groups that fit a warp, that do not, and that no vector load divides; large and tiny states against eps."""
    cfg = dh.config(48, 60, [dh.retention(2, 8, group, (0.9, 0.99)), dh.parallel(dh.attention(1, 1, 8, 8, 8), dh.state(1, 8, dim, (0.9,)))], eps=1e-3)
    ids = np.arange(24)
    for gain in (1.0, 0.02):
        W = dh.weights(cfg, 43)
        for n in ("l0.mix.v", "l1.mix.right.v"):
            W[n] = dh.bf16_round(W[n] * gain)
        want = do.forward(W, cfg, ids, want_layers=True)[1]
        m = make(cfg, W, dtype)
        c = make.cache(m)
        for cut in (8192, 4, 1):
            c.reset()
            got = m.step_layers(c, ids, prefill_step=cut)
            assert dh.rel(got, want) < TOL[dtype], (gain, cut, dh.rel(got, want))


# ------------------------------------------------------------------ single keys that must be seen
def needle_model(kind):
    """Token 1 leaves a key that token 2's query singles out at any distance: both lie along one entry that does not
    turn.  kind: the mechanism that has to find it."""
    if kind == "left":
        cfg = dh.config(128, 64, [dh.parallel(dh.attention(4, 2, 32, 24, 16, scale=0.4, softcap=30.0), dh.state(1, 8, 8, (0.5,)))], alpha=0.1)
        p, heads, dim, e = "l0.mix.left.", 4, 32, 20
    elif kind == "right":
        cfg = dh.config(128, 64, [dh.parallel(dh.attention(1, 1, 8, 8, 8), dh.state(2, 24, 16, (0.9995, 0.99975)))], alpha=0.1)
        p, heads, dim, e = "l0.mix.right.", 2, 24, 5
    else:
        cfg = dh.config(128, 64, [dh.retention(2, 24, 16, (0.9995, 0.99975), rot_dims=8)], alpha=0.1)
        p, heads, dim, e = "l0.mix.", 2, 24, 20
    W = silence(cfg, dh.weights(cfg, 51), [kind])
    dual = np.linalg.pinv(W["embed"].astype(np.float64) * cfg["embedding"]["scale"])  # column j reads token j and no other
    gain = 60.0 if kind == "left" else 25.0
    for h in range(heads):
        kv = h // 2 if kind == "left" else h
        q, k = W[p + "q"], W[p + "k"]
        if kind != "left":  # noise tokens leave little
            k[kv * dim:(kv + 1) * dim] *= 0.05
        q[h * dim + e] = gain * dual[:, 2]
        k[kv * dim + e] = gain * dual[:, 1]
    for n in ("q", "k"):
        W[p + n] = dh.bf16_round(W[p + n])
    return cfg, W


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", ["left", "right", "retention"])
def test_a_far_key_is_found_wherever_it_lies(make, kind, dtype):
    """The key at the first places, at the edges of key tiles, key ranges and state chunks, and right before the
    query; the query in a prompt chunk, in a short portion and decoded alone.  Taking the key away changes the
    answer by far more than the tolerance."""
    T = 400
    cfg, W = needle_model(kind)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    noise = np.random.default_rng(8).integers(3, cfg["vocab"], T)
    noise[-1] = 2
    without = do.forward(W, cfg, noise)[-1]
    for at in (0, 1, 2, 31, 32, 33, 63, 64, 65, 127, 128, 191, 192, 255, 256, 257, 319, 320, 383, 384, T - 3, T - 2):
        ids = noise.copy()
        ids[at] = 1
        want = do.forward(W, cfg, ids)[-1]
        assert dh.rel(without, want) > 5 * TOL[dtype], ("the key does not matter enough to test anything", dh.rel(without, want))
        for cut in ((T,), (T - 1, 1), (T - 2, 2), (T - 20, 20), (T - 70, 70)):
            c.reset()
            for j, n in enumerate(cut):
                lo = sum(cut[:j])
                lg = m.step(c, ids[lo:lo + n], [n - 1])
            assert dh.rel(lg[0], want) < TOL[dtype], (at, cut, dh.rel(lg[0], want))


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", ["left", "right", "retention"])
def test_the_mask_ends_at_the_row_itself(make, kind, dtype):
    """The singled-out key one place after the query is not seen, one before it is: in chunks the causal edge runs
    through every tile."""
    T = 300
    cfg, W = needle_model(kind)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    rng = np.random.default_rng(9)
    for q in (5, 15, 16, 31, 32, 63, 64, 100, 255, 256):
        ids = rng.integers(3, cfg["vocab"], T)
        ids[q], ids[q + 1], ids[q + 2] = 2, 1, 2
        want = do.forward(W, cfg, ids)
        for cut in (8192, 33, 16, 4):
            c.reset()
            lg = m.step(c, ids, [q, q + 1, q + 2], prefill_step=cut)
            assert dh.rel(lg, want[q:q + 3]) < TOL[dtype], (q, cut)


# ------------------------------------------------------------------ cuts, reuse, long decoding
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name,T", [("mixed", 330), ("odd", 140), ("wide", 290)])
def test_portions_of_every_size_agree(make, name, T, dtype):
    cfg, W, ids, logits, _ = oracle(name, 7, T)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    whole = m.step(c, ids, range(T))
    for size in (1, 2, 3, 4, 5, 6, 16, 31, 32, 33, 63, 64, 65, 128, 256, 257):
        c.reset()
        rows = [m.step(c, ids[lo:lo + size], range(len(ids[lo:lo + size]))) for lo in range(0, T, size)]
        got = np.concatenate(rows)
        assert dh.rel(got, whole) < SAME[dtype], (size, dh.rel(got, whole))
        per_row = np.sqrt(((got - logits) ** 2).mean(-1)) / np.sqrt((logits ** 2).mean())
        assert per_row.max() < 3 * TOL[dtype], (size, int(per_row.argmax()), per_row.max())


@pytest.mark.parametrize("dtype", DT)
def test_wanted_rows_are_the_same_rows(make, dtype):
    cfg, W, ids, logits, _ = oracle("mixed", 7, 330)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    full = m.step(c, ids, range(330))
    for want in ([], [0], [329], [3, 4, 77], [328, 329]):
        c.reset()
        got = m.step(c, ids, want, prefill_step=64)
        assert got.shape == (len(want), cfg["vocab"])
        if want:
            assert dh.rel(got, full[want]) < SAME[dtype]


@pytest.mark.parametrize("dtype", DT)
def test_requests_side_by_side_equal_each_alone(make, dtype):
    """Unequal requests whose portions and single tokens alternate, each on its own cache: the bits of each alone."""
    cfg = dh.CONFIGS["mixed"]
    m = make(cfg, dh.weights(cfg, 7), dtype)
    rng = np.random.default_rng(12)
    reqs = [rng.integers(0, cfg["vocab"], n) for n in (90, 7, 41)]
    cuts = [[50, 2, 30, 1, 1, 6], [1, 1, 1, 1, 1, 2], [4, 5, 1, 1, 10, 20]]
    caches = [make.cache(m) for _ in reqs]

    def portion(r, j):
        lo = sum(cuts[r][:j])
        return reqs[r][lo:lo + cuts[r][j]]

    together = [[None] * 6 for _ in reqs]
    for j in range(6):
        for r in (2, 0, 1):
            ids = portion(r, j)
            together[r][j] = m.step(caches[r], ids, range(len(ids)))
    for r in range(3):
        caches[0].reset()  # also a cache that another request has used
        for j in range(6):
            ids = portion(r, j)
            assert np.array_equal(m.step(caches[0], ids, range(len(ids))), together[r][j]), (r, j)


@pytest.mark.parametrize("dtype", DT)
def test_a_used_cache_is_as_good_as_a_new_one(make, dtype):
    """After a long request a short one on the same cache: no state and no key of the old one is left."""
    for name in ("odd", "mixed"):
        cfg = dh.CONFIGS[name]
        m = make(cfg, dh.weights(cfg, 7), dtype)
        rng = np.random.default_rng(13)
        old, new = rng.integers(0, cfg["vocab"], 300), rng.integers(0, cfg["vocab"], 45)
        c, fresh = make.cache(m), make.cache(m)
        m.step(c, old, [299])
        for t in old[:7]:
            m.step(c, [t], [])  # the state ring has turned
        c.reset()
        a = [m.step(c, new[:40], range(40)), m.step(c, new[40:41], [0]), m.step(c, new[41:], range(4))]
        b = [m.step(fresh, new[:40], range(40)), m.step(fresh, new[40:41], [0]), m.step(fresh, new[41:], range(4))]
        for x, y in zip(a, b):
            assert np.array_equal(x, y)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_windows_can_be_taken_back(make, name, dtype):
    """A captured window of which some rows are kept: keys and states that follow equal never having run the rest."""
    cfg = dh.CONFIGS[name]
    m = make(cfg, dh.weights(cfg, 7), dtype)
    a, b = make.cache(m), make.cache(m)
    ids = np.arange(40) * 7 % cfg["vocab"]
    for keep, rows in ((1, 2), (2, 4), (3, 4), (4, 4), (1, 4)):
        a.reset()
        b.reset()
        for c in (a, b):
            m.step(c, ids[:20], [])
        for lap in range(3):  # the ring turns over
            lo = 20 + lap * keep
            win = np.concatenate([ids[lo:lo + keep], [3, 4, 5]])[:rows]
            m.forward(a, win, capture=True)
            a.rewind(keep)
            m.forward(b, ids[lo:lo + keep])
        assert a.offset == b.offset == 20 + 3 * keep
        x, y = m.step(a, ids[32:], range(8)), m.step(b, ids[32:], range(8))
        assert dh.rel(x, y) < SAME[dtype], (keep, rows)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_generation_loop(pkg, make, name, dtype):
    """Long decoding through generate_step (graphs, programmatic launches, device-side sampling): every token is the
    oracle's argmax for what came before it, up to ties within the tolerance."""
    cfg = dh.CONFIGS[name]
    W = dh.weights(cfg, 7)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    for prompt_len, n in ((1, 40), (3, 20), (60, 300)):
        prompt = np.random.default_rng(prompt_len).integers(0, cfg["vocab"], prompt_len)
        c.reset()
        out = pkg.generate_step(m, c, prompt, n)
        assert len(out) == n and c.offset == prompt_len + n
        ids = np.concatenate([prompt, out])
        logits = do.forward(W, cfg, ids)[prompt_len - 1:-1]
        slack = 8 * TOL[dtype] * np.sqrt((logits ** 2).mean())
        gap = logits.max(-1) - logits[np.arange(n), out]
        assert gap.max() <= slack, (prompt_len, int(gap.argmax()), gap.max())
        if dtype == "float32":
            assert (gap > 0).mean() < 0.02
        c.reset()
        assert pkg.generate_step(m, c, prompt, n) == out  # the captured steps replay to the same tokens


def test_greedy_equals_step_by_step_argmax(pkg, make):
    cfg = dh.CONFIGS["wide"]
    m = make(cfg, dh.weights(cfg, 7), "bfloat16")
    c = make.cache(m)
    prompt = np.arange(50)
    out = pkg.generate_step(m, c, prompt, 12)
    c.reset()
    lg = m.step(c, prompt, [49])
    for t in out:
        top = np.sort(lg[0])[-2:]
        assert int(lg[0].argmax()) == t or top[1] - top[0] < 0.02 * np.abs(lg).max()
        lg = m.step(c, [t], [0])


def test_hidden_rows_and_head(make):
    """forward / prefill hand out rows after the final norm; head_greedy takes them."""
    cfg, W, ids, logits, _ = oracle("odd", 7, 140)
    for dtype in DT:
        m = make(cfg, W, dtype)
        c = make.cache(m)
        hid = m.prefill(c, ids[:30], want_hidden=True)
        assert hid.numpy().shape == (30, 104)
        last = m.forward(c, ids[30:32])
        toks, lg = m.head_greedy(last, 2, want_logits=True)
        lg = lg.numpy()
        assert dh.rel(lg, logits[30:32]) < TOL[dtype]
        assert list(toks) == list(lg.argmax(-1))


# ------------------------------------------------------------------ control path
CONTROL = """
import sys, numpy as np
sys.path[:0] = [%r, %r]
import __graft_entry__ as g
pkg = g.load_package()
ctx = pkg.Context(0)
m = pkg.TextModel.load(ctx, sys.argv[1], max_ctx=512)
c = m.make_cache()
ids = np.load(sys.argv[2])
a = m.step(c, ids[:-9], range(len(ids) - 9))
b = [m.step(c, ids[i:i + 1], [0]) for i in range(len(ids) - 9, len(ids))]
np.save(sys.argv[3], np.concatenate([a] + b))
"""


@pytest.mark.parametrize("name,T", [("mixed", 330), ("odd", 140)])
def test_one_kernel_per_operation_agrees(tmp_path, name, T):
    """ORN_UNFUSED=1 (bfloat16, plain kernels) against the fused and tensor-core routes."""
    cfg, W, ids, logits, _ = oracle(name, 7, T)
    path = dh.write_artifact(tmp_path / "m", cfg, W, skew=1)
    np.save(tmp_path / "ids.npy", ids)
    got = {}
    for mode in ("0", "1"):
        out = str(tmp_path / ("o%s.npy" % mode))
        subprocess.run([sys.executable, "-c", CONTROL % (ROOT, os.path.join(ROOT, "tests")), path, str(tmp_path / "ids.npy"), out],
                       check=True, timeout=300, env=dict(os.environ, ORN_UNFUSED=mode))
        got[mode] = np.load(out)
        assert dh.rel(got[mode], logits) < TOL["bfloat16"]
    assert dh.rel(got["0"], got["1"]) < SAME["bfloat16"]


# ------------------------------------------------------------------ registry, loader, limits
def test_configurations_that_are_refused(pkg, ctx):
    ok = small()
    pkg.TextModel.from_config(ctx, ok).free()

    def bad(change):
        cfg = json.loads(json.dumps(ok))
        change(cfg)
        with pytest.raises(pkg.OrnError):
            pkg.TextModel.from_config(ctx, cfg)

    mix = lambda c, i: c["layers"][i]["mixer"]  # noqa: E731
    bad(lambda c: c.pop("width"))
    bad(lambda c: c.pop("postln_alpha"))
    bad(lambda c: c.pop("embedding"))
    bad(lambda c: c.update(layers=[]))
    bad(lambda c: c["layers"][0].update(type="latent_attention"))
    bad(lambda c: c["layers"][0].update(mixer=None))
    bad(lambda c: mix(c, 0).pop("right"))
    bad(lambda c: mix(c, 0)["left"].update(kv_heads=3))
    bad(lambda c: mix(c, 0)["left"].update(heads=0))
    bad(lambda c: mix(c, 0)["left"].pop("scale"))
    bad(lambda c: mix(c, 0)["left"].update(softcap=-1.0))
    bad(lambda c: mix(c, 0)["left"]["rot"].update(dims=18))
    bad(lambda c: mix(c, 0)["right"].update(decay=[0.5]))
    bad(lambda c: mix(c, 1).update(decay=[0.5, 1.5]))
    bad(lambda c: mix(c, 1)["rot"].update(dims=3))
    bad(lambda c: c["layers"][0]["mlp"].update(kind="routed"))


def test_artifacts_that_are_refused(pkg, ctx, tmp_path):
    cfg = small()
    W = dh.weights(cfg, 1)
    for i, change in enumerate([lambda w: w.pop("l0.mix.left.sink"), lambda w: w.update({"l1.norm1": w["l1.norm1"][:-1]}),
                                lambda w: w.update({"embed": w["embed"][:, :-1]})]):
        bad = dict(W)
        change(bad)
        with pytest.raises(pkg.OrnError):
            pkg.TextModel.load(ctx, dh.write_artifact(tmp_path / str(i), cfg, bad))


def test_limits_are_errors(pkg, make):
    cfg = small()
    m = make(cfg, dh.weights(cfg, 1), "bfloat16", max_ctx=16)
    c = make.cache(m)
    with pytest.raises(pkg.OrnError):
        m.step(c, np.zeros(17, np.uint32), [])
    c.reset()
    with pytest.raises(pkg.OrnError):
        m.step(c, [cfg["vocab"]], [0])
    with pytest.raises(pkg.OrnError):
        pkg.Batch(m, 2)
    with pytest.raises(pkg.OrnError):
        pkg.generate_step_mtp(m, c, [1, 2], 1, 4)
    assert m.step(c, np.arange(16), [15]).shape == (1, cfg["vocab"])
    with pytest.raises(pkg.OrnError):
        m.step(c, [1], [0])


def test_random_weights_and_names(pkg, ctx):
    """A model from its configuration alone; matrices come back under their names."""
    cfg = dh.config(128, 96, [dh.retention(2, 16, 24, (0.9, 0.99), ff=64), dh.parallel(dh.attention(4, 2, 16, 24, 8), dh.state(2, 24, 16, (0.9, 0.95)))])
    m = pkg.TextModel.from_config(ctx, cfg, max_ctx=64)
    m.init_random(5)
    W = {}
    for name, shape in dh.tensors(cfg).items():
        w = m.get_linear(name).export()[0].view(np.uint16) if len(shape) == 2 else m.get_tensor(name)
        W[name] = (w.astype(np.uint32) << 16).view(np.float32).reshape(shape)
    assert m.weight_bytes() == 2 * sum(w.size for w in W.values())
    c = m.make_cache()
    ids = np.arange(40)
    assert dh.rel(m.step(c, ids, range(40)), do.forward(W, cfg, ids)) < TOL["bfloat16"]
    c.free()
    m.free()


# ------------------------------------------------------------------ trace replay
@pytest.mark.parametrize("dtype", DT)
def test_trace_replay_program(tmp_path, dtype):
    """bin/trace_run over requests that follow and overlap one another, with caches given back and used again;
    answers compared with the plain implementation."""
    cfg = dh.CONFIGS["mixed"]
    W = dh.weights(cfg, 7)
    path = dh.write_artifact(tmp_path / "m", cfg, W)
    rng = np.random.default_rng(3)
    req = {k: rng.integers(0, cfg["vocab"], n).tolist() for k, n in (("a", 50), ("b", 9), ("c", 33))}
    plan = [("a", 30, [0, 29]), ("b", 9, [8, 2]), ("a", 2, [1]), ("a", 1, []), ("a", 17, [16]), ("c", 1, [0]), ("c", 32, [5, 31])]
    at = dict.fromkeys(req, 0)
    lines, expect = [], {}
    for n, (r, count, want) in enumerate(plan):
        lo, at[r] = at[r], at[r] + count
        end = [r] if at[r] == len(req[r]) else []
        lines.append(json.dumps({"step": n, "entries": [{"id": r, "tokens": req[r][lo:lo + count], "want": want}], "end": end}))
        if want:
            expect[n] = (r, [lo + w for w in want])
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                       input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.split("\n") if x.startswith("done")] == ["done %d" % i for i in range(len(plan))]
    full = {r: do.forward(W, cfg, ids) for r, ids in req.items()}
    for n, (r, places) in expect.items():
        got = np.fromfile(out / ("%d.f32" % n), "<f4").reshape(len(places), cfg["vocab"])
        assert dh.rel(got, full[r][places]) < TOL[dtype], (n, r)
