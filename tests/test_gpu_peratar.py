"""The Peratar decoder on the GPU against the plain numpy implementation (oracle/peratar_oracle.py).

float32 models are held to rounding in float32, bfloat16 ones to rounding of activations; both are
compared at every layer where the difference would show first."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import peratar_helpers as ph
import peratar_oracle as po

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 3e-2}   # rms of the difference over rms of the value
SAME = {"float32": 5e-6, "bfloat16": 3e-2}  # the same positions reached by another cut


@pytest.fixture(scope="module")
def make(pkg, ctx, tmp_path_factory):
    """(config, weights, dtype) -> a loaded model; models and caches are freed with the module."""
    made = []

    def build(cfg, W, dtype, max_ctx=512):
        path = ph.write_artifact(tmp_path_factory.mktemp("m"), cfg, W)
        m = pkg.TextModel.load(ctx, path, max_ctx=max_ctx, dtype=pkg.DT_F32 if dtype == "float32" else pkg.DT_BF16)
        made.append(m)
        return m

    caches = []

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
        cfg = ph.CONFIGS[name]
        W = ph.weights(cfg, seed)
        ids = np.random.default_rng(seed + 1000).integers(0, cfg["vocab"], T)
        _ORACLE[key] = (cfg, W, ids) + po.forward(W, cfg, ids, want_layers=True)
    return _ORACLE[key]


DT = ["float32", "bfloat16"]


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name,T", [("mixed", 150), ("odd", 140), ("one", 60), ("unrotated", 90), ("wide", 100), ("edges", 90)])
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
            assert ph.rel(got[i], streams[i, :n]) < TOL[dtype], (cut, "layer", i, ph.rel(got[i], streams[i, :n]))
        c.reset()
        lg = m.step(c, ids[:n], range(n), prefill_step=cut)
        assert ph.rel(lg, logits[:n]) < TOL[dtype], (cut, ph.rel(lg, logits[:n]))


# ------------------------------------------------------------------ one mechanism at a time
def silence(cfg, W, keep):
    """Weights under which only the mechanisms in `keep` act: a zero norm weight removes a sublayer, a
    large gate bias opens its gate, averaging weights (0, .., 0, 1) pass the newest stream on."""
    W = {k: v.copy() for k, v in W.items()}
    for k in W:
        if k.endswith("norm1") and "mixer" not in keep:
            W[k][:] = 0
        if k.endswith("norm2") and "ff" not in keep:
            W[k][:] = 0
        if ".rg" in k and "gate" not in keep:
            W[k][:] = 30 if k.endswith(".b") else 0
        if k.endswith("dwa") and "average" not in keep:
            W[k][:] = 0
            W[k][-1] = 1
    return W


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("keep", [["mixer"], ["ff"], ["average"], ["mixer", "gate"], ["ff", "gate"], ["ff", "average"]], ids="+".join)
def test_one_mechanism_alone(make, keep, dtype):
    cfg = ph.CONFIGS["mixed"]
    W = silence(cfg, ph.weights(cfg, 21), keep)
    ids = np.random.default_rng(5).integers(0, cfg["vocab"], 70)
    want = po.forward(W, cfg, ids, want_layers=True)[1]
    m = make(cfg, W, dtype)
    c = make.cache(m)
    for cut in (8192, 3):
        c.reset()
        got = m.step_layers(c, ids, prefill_step=cut)
        for i in range(len(want)):
            assert ph.rel(got[i], want[i]) < TOL[dtype], (keep, cut, i)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("p,q", [(-4.0, 3.0), (3.0, -4.0), (0.0, 0.0)])
def test_xielu_both_sides(make, p, q, dtype):
    """The two learned numbers far apart and equal, pre-activations on both sides of zero and large."""
    cfg = ph.config(64, 80, [ph.layer(ph.mixer(2, 8, 4, 8, 16), 48)])
    W = silence(cfg, ph.weights(cfg, 31), ["ff"])
    W["l0.mlp.act"][:] = [p, q]
    W["l0.mlp.up"] *= 4
    ids = np.arange(60)
    want = po.forward(W, cfg, ids, want_layers=True)[1]
    m = make(cfg, W, dtype)
    c = make.cache(m)
    for cut in (8192, 2):
        c.reset()
        assert ph.rel(m.step_layers(c, ids, prefill_step=cut), want) < TOL[dtype]


def test_norm_eps_and_softcap_are_read(make):
    """A large eps and a small cap: both change the result visibly, and the result follows."""
    base = ph.config(64, 80, [ph.layer(ph.mixer(2, 8, 4, 8, 16), 48)], eps=1e-6, softcap=50.0)
    W = ph.weights(base, 41)
    ids = np.arange(20)
    plain = po.forward(W, base, ids)
    for change in ({"norm": {"eps": 0.5}}, {"logit_softcap": 1.5}):
        cfg = dict(base, **change)
        want = po.forward(W, cfg, ids)
        assert ph.rel(want, plain) > 100 * TOL["float32"]
        for dtype in DT:
            m = make(cfg, W, dtype)
            assert ph.rel(m.step(make.cache(m), ids, range(20)), want) < TOL[dtype]


# ------------------------------------------------------------------ attention: single keys that must be seen
def needle_model(T_max, sharp=14.0):
    """Token 1 is a key that token 2's query singles out (score `sharp` above the rest, whatever the
    distance: that head's rotated query is zero); everything else is noise."""
    cfg = ph.config(128, 64, [ph.layer(ph.mixer(2, 16, 8, 24, 32), 64), ph.layer(ph.mixer(3, 8, 8, 16, 32, kv_from=0), None)])
    W = ph.weights(cfg, 51, q_gain=0.5)
    for i, d in ((0, 16), (1, 8)):
        m = cfg["layers"][i]["mixer"]
        c = po.rms_norm(W["l0.mix.dkv"][:32] @ W["embed"][1], W["l0.mix.dkv.norm"], cfg["norm"]["eps"])
        k = W["l%d.mix.uk" % i][:d] @ c
        b = W["embed"][2]
        q = W["l%d.mix.q" % i]
        q[:d + 8] = 0
        q[:d] = np.outer(k / (k @ k), b / (b @ b)) * sharp / m["scale"]
        W["l%d.mix.q" % i] = ph.bf16_round(q)
    W["l0.dwa"] = np.array([0.0, 1.0], np.float32)
    return cfg, W


@pytest.mark.parametrize("dtype", DT)
def test_a_far_key_is_found_wherever_it_lies(make, dtype):
    """The key at the first places, at the edges of the kernels' key tiles and key ranges, and right
    before the query; the query in a prompt chunk, in a short portion and decoded alone.  Taking the key
    away changes the answer by far more than the tolerance."""
    T = 400
    cfg, W = needle_model(T)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    rng = np.random.default_rng(8)
    noise = rng.integers(3, cfg["vocab"], T)
    noise[-1] = 2
    without = po.forward(W, cfg, noise)[-1]
    for at in (0, 1, 2, 31, 32, 33, 63, 64, 65, 127, 128, 191, 192, 255, 256, 319, 320, 383, 384, T - 3, T - 2):
        ids = noise.copy()
        ids[at] = 1
        want = po.forward(W, cfg, ids)[-1]
        assert ph.rel(without, want) > 5 * TOL[dtype], "the key does not matter enough to test anything"
        for cut in ((T,), (T - 1, 1), (T - 2, 2), (T - 20, 20), (T - 70, 70)):
            c.reset()
            for j, n in enumerate(cut):
                lo = sum(cut[:j])
                lg = m.step(c, ids[lo:lo + n], [n - 1])
            assert ph.rel(lg[0], want) < TOL[dtype], (at, cut, ph.rel(lg[0], want))


@pytest.mark.parametrize("dtype", DT)
def test_the_mask_ends_at_the_row_itself(make, dtype):
    """The singled-out key one place after the query is not seen, at the query's own place and one before
    it is: in chunks the causal edge runs through every tile."""
    T = 140
    cfg, W = needle_model(T)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    rng = np.random.default_rng(9)
    for q in (5, 15, 16, 31, 32, 63, 64, 100):
        ids = rng.integers(3, cfg["vocab"], T)
        ids[q], ids[q + 1] = 2, 1
        want = po.forward(W, cfg, ids)
        for cut in (8192, 33, 16, 4):
            c.reset()
            lg = m.step(c, ids, [q, q + 1], prefill_step=cut)
            assert ph.rel(lg, want[[q, q + 1]]) < TOL[dtype], (q, cut)


# ------------------------------------------------------------------ cuts, reuse, long decoding
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_portions_of_every_size_agree(make, name, dtype):
    T = 139
    cfg, W, ids, logits, _ = oracle(name, 7, T)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    whole = m.step(c, ids, range(T))
    for size in (1, 2, 3, 4, 5, 6, 16, 31, 32, 33, 63, 64, 65, 128):
        c.reset()
        rows = [m.step(c, ids[lo:lo + size], range(len(ids[lo:lo + size]))) for lo in range(0, T, size)]
        got = np.concatenate(rows)
        assert ph.rel(got, whole) < SAME[dtype], (size, ph.rel(got, whole))
        per_row = np.sqrt(((got - logits) ** 2).mean(-1)) / np.sqrt((logits ** 2).mean())
        assert per_row.max() < 3 * TOL[dtype], (size, int(per_row.argmax()), per_row.max())


@pytest.mark.parametrize("dtype", DT)
def test_wanted_rows_are_the_same_rows(make, dtype):
    cfg, W, ids, logits, _ = oracle("mixed", 7, 150)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    full = m.step(c, ids, range(150))
    for want in ([], [0], [149], [3, 4, 77], [148, 149]):
        c.reset()
        got = m.step(c, ids, want, prefill_step=64)
        assert got.shape == (len(want), cfg["vocab"])
        if want:
            assert ph.rel(got, full[want]) < SAME[dtype]


@pytest.mark.parametrize("dtype", DT)
def test_requests_side_by_side_equal_each_alone(make, dtype):
    """Unequal requests whose portions and single tokens alternate, each on its own cache: the bits of
    each alone."""
    cfg = ph.CONFIGS["mixed"]
    m = make(cfg, ph.weights(cfg, 7), dtype)
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
    """After a long request a short one on the same cache, and after growing chunks a small one."""
    cfg = ph.CONFIGS["odd"]
    m = make(cfg, ph.weights(cfg, 7), dtype)
    rng = np.random.default_rng(13)
    old, new = rng.integers(0, cfg["vocab"], 300), rng.integers(0, cfg["vocab"], 45)
    c, fresh = make.cache(m), make.cache(m)
    m.step(c, old, [299])
    c.reset()
    a = [m.step(c, new[:40], range(40)), m.step(c, new[40:41], [0]), m.step(c, new[41:], range(4))]
    b = [m.step(fresh, new[:40], range(40)), m.step(fresh, new[40:41], [0]), m.step(fresh, new[41:], range(4))]
    for x, y in zip(a, b):
        assert np.array_equal(x, y)


def test_windows_can_be_taken_back(make):
    """A captured window of four rows of which two are kept: what follows equals never having run them."""
    cfg = ph.CONFIGS["mixed"]
    W = ph.weights(cfg, 7)
    for dtype in DT:
        m = make(cfg, W, dtype)
        a, b = make.cache(m), make.cache(m)
        ids = np.arange(30) * 7 % cfg["vocab"]
        for c in (a, b):
            m.step(c, ids[:20], [])
        m.forward(a, np.array([ids[20], ids[21], 3, 4]), capture=True)
        a.rewind(2)
        m.forward(b, ids[20:22])
        assert a.offset == b.offset == 22
        x, y = m.step(a, ids[22:], range(8)), m.step(b, ids[22:], range(8))
        assert ph.rel(x, y) < SAME[dtype]


@pytest.mark.parametrize("dtype", DT)
def test_greedy_generation_through_the_generation_loop(pkg, make, dtype):
    """Long decoding through generate_step (graphs, programmatic launches, device-side sampling): every
    token is the oracle's argmax for what came before it, up to ties within the tolerance."""
    cfg = ph.CONFIGS["mixed"]
    W = ph.weights(cfg, 7)
    m = make(cfg, W, dtype)
    c = make.cache(m)
    for prompt_len, n in ((1, 40), (3, 20), (60, 300)):
        prompt = np.random.default_rng(prompt_len).integers(0, cfg["vocab"], prompt_len)
        c.reset()
        out = pkg.generate_step(m, c, prompt, n)
        assert len(out) == n and c.offset == prompt_len + n
        ids = np.concatenate([prompt, out])
        logits = po.forward(W, cfg, ids)[prompt_len - 1:-1]
        slack = 8 * TOL[dtype] * np.sqrt((logits ** 2).mean())
        gap = logits.max(-1) - logits[np.arange(n), out]
        assert gap.max() <= slack, (prompt_len, int(gap.argmax()), gap.max())
        if dtype == "float32":
            assert (gap > 0).mean() < 0.02
        c.reset()
        assert pkg.generate_step(m, c, prompt, n) == out  # the captured steps replay to the same tokens


def test_greedy_equals_step_by_step_argmax(pkg, make):
    cfg = ph.CONFIGS["wide"]
    m = make(cfg, ph.weights(cfg, 7), "bfloat16")
    c = make.cache(m)
    prompt = np.arange(50)
    out = pkg.generate_step(m, c, prompt, 12)
    c.reset()
    lg = m.step(c, prompt, [49])
    for t in out:
        top = np.sort(lg[0])[-2:]
        assert int(lg[0].argmax()) == t or top[1] - top[0] < 0.02
        lg = m.step(c, [t], [0])


def test_hidden_rows_and_head(make):
    """forward / prefill hand out rows after the final norm; head_greedy takes them."""
    cfg, W, ids, logits, _ = oracle("odd", 7, 140)
    for dtype in DT:
        m = make(cfg, W, dtype)
        c = make.cache(m)
        hid = m.prefill(c, ids[:30], want_hidden=True)
        rows = hid.numpy()
        assert rows.shape == (30, 104)
        last = m.forward(c, ids[30:32])
        toks, lg = m.head_greedy(last, 2, want_logits=True)
        lg = lg.numpy()
        assert ph.rel(lg, logits[30:32]) < TOL[dtype]
        assert list(toks) == list(lg.argmax(-1))


# ------------------------------------------------------------------ control path
CONTROL = """
import sys, numpy as np
sys.path[:0] = [%r, %r]
import __graft_entry__ as g
pkg = g.load_package()
ctx = pkg.Context(0)
m = pkg.TextModel.load(ctx, sys.argv[1], max_ctx=256)
c = m.make_cache()
ids = np.load(sys.argv[2])
a = m.step(c, ids[:-9], range(len(ids) - 9))
b = [m.step(c, ids[i:i + 1], [0]) for i in range(len(ids) - 9, len(ids))]
np.save(sys.argv[3], np.concatenate([a] + b))
"""


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_one_kernel_per_operation_agrees(make, tmp_path, name):
    """ORN_UNFUSED=1 (bfloat16, plain kernels) against the fused and tensor-core routes."""
    cfg, W, ids, logits, _ = oracle(name, 7, 139)
    path = ph.write_artifact(tmp_path / "m", cfg, W, skew=1)
    np.save(tmp_path / "ids.npy", ids)
    got = {}
    for mode in ("0", "1"):
        out = str(tmp_path / ("o%s.npy" % mode))
        subprocess.run([sys.executable, "-c", CONTROL % (ROOT, os.path.join(ROOT, "tests")), path, str(tmp_path / "ids.npy"), out],
                       check=True, timeout=300, env=dict(os.environ, ORN_UNFUSED=mode))
        got[mode] = np.load(out)
        assert ph.rel(got[mode], logits) < TOL["bfloat16"]
    assert ph.rel(got["0"], got["1"]) < SAME["bfloat16"]


# ------------------------------------------------------------------ registry, loader, limits
def test_configurations_that_are_refused(pkg, ctx):
    ok = ph.CONFIGS["one"]
    pkg.TextModel.from_config(ctx, ok).free()

    def bad(change):
        cfg = json.loads(json.dumps(ok))
        change(cfg)
        with pytest.raises(pkg.OrnError):
            pkg.TextModel.from_config(ctx, cfg)

    bad(lambda c: c.update(architecture="Other"))
    bad(lambda c: c.pop("width"))
    bad(lambda c: c.update(layers=[]))
    bad(lambda c: c["layers"][0].update(type="convolution"))
    bad(lambda c: c["layers"][0]["mixer"].update(kv_from=0))
    bad(lambda c: c["layers"][0]["mixer"].update(heads=0))
    bad(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3))
    bad(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4))
    bad(lambda c: c["layers"][0]["mlp"].update(kind="routed"))
    bad(lambda c: c["layers"].append(ph.layer(ph.mixer(1, 8, 2, 8, 16, kv_from=0), None)))
    with pytest.raises(pkg.OrnError):
        pkg.TextModel.from_config(ctx, ok, dtype=7)


def test_artifacts_that_are_refused(pkg, ctx, tmp_path):
    cfg = ph.CONFIGS["one"]
    W = ph.weights(cfg, 1)
    for i, change in enumerate([lambda w: w.pop("l0.mix.g"), lambda w: w.update({"l0.dwa": w["l0.dwa"][:1]}),
                                lambda w: w.update({"head": w["head"][:, :-1]})]):
        bad = dict(W)
        change(bad)
        with pytest.raises(pkg.OrnError):
            pkg.TextModel.load(ctx, ph.write_artifact(tmp_path / str(i), cfg, bad))


def test_limits_are_errors(pkg, ctx, make):
    cfg = ph.CONFIGS["one"]
    m = make(cfg, ph.weights(cfg, 1), "bfloat16", max_ctx=16)
    c = make.cache(m)
    with pytest.raises(pkg.OrnError):
        m.step(c, np.zeros(17, np.uint32), [])
    c.reset()
    with pytest.raises(pkg.OrnError):
        m.step(c, [cfg["vocab"]], [0])
    with pytest.raises(pkg.OrnError):
        m.step(c, [1, 2], [1, 0])
    with pytest.raises(pkg.OrnError):
        m.step(c, [1, 2], [2])
    with pytest.raises(pkg.OrnError):
        pkg.Batch(m, 2)
    with pytest.raises(pkg.OrnError):
        pkg.generate_step_mtp(m, c, [1, 2], 1, 4)
    assert m.step(c, np.arange(16), [15]).shape == (1, cfg["vocab"])
    with pytest.raises(pkg.OrnError):
        m.step(c, [1], [0])


def test_random_weights_and_names(pkg, ctx):
    """A model from its configuration alone; matrices come back under their names."""
    cfg = ph.config(128, 96, [ph.layer(ph.mixer(2, 16, 8, 16, 32), 64)])
    m = pkg.TextModel.from_config(ctx, cfg, max_ctx=64)
    m.init_random(5)
    W = {}
    for name, shape in ph.tensors(cfg).items():
        if len(shape) == 2:
            w = m.get_linear(name).export()[0].view(np.uint16)
        else:
            w = m.get_tensor(name)
        W[name] = (w.astype(np.uint32) << 16).view(np.float32).reshape(shape)
    assert m.weight_bytes() == 2 * sum(w.size for w in W.values())
    c = m.make_cache()
    ids = np.arange(40)
    assert ph.rel(m.step(c, ids, range(40)), po.forward(W, cfg, ids)) < TOL["bfloat16"]
    c.free()
    m.free()


# ------------------------------------------------------------------ trace replay
@pytest.mark.parametrize("dtype", DT)
def test_trace_replay_program(make, tmp_path, dtype):
    """bin/trace_run over requests that follow and overlap one another, with caches given back and used
    again; answers compared with the plain implementation."""
    cfg = ph.CONFIGS["mixed"]
    W = ph.weights(cfg, 7)
    path = ph.write_artifact(tmp_path / "m", cfg, W)
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
    assert sorted(os.listdir(out)) == sorted("%d.f32" % n for n in expect)
    full = {r: po.forward(W, cfg, ids) for r, ids in req.items()}
    for n, (r, places) in expect.items():
        got = np.fromfile(out / ("%d.f32" % n), "<f4").reshape(len(places), cfg["vocab"])
        assert ph.rel(got, full[r][places]) < TOL[dtype], (n, r)
