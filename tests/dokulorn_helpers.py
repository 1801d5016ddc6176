"""Small Dokulorn models with random weights for the tests: configuration and weights."""
import numpy as np

from peratar_helpers import bf16_round, rel, write_artifact  # noqa: F401  (artifacts have one format)


def rot(dims, base=10000.0):
    return {"base": base, "dims": dims}


def retention(heads, dim, vdim, decay, rot_dims=None, base=10000.0, ff=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": rot(dim if rot_dims is None else rot_dims, base)}
    return {"type": "retention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def attention(heads, kv_heads, dim, vdim, rot_dims, base=10000.0, scale=None, softcap=20.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot(rot_dims, base),
            "scale": dim ** -0.5 if scale is None else scale, "softcap": softcap}


def state(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def parallel(left, right, ff=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, eps=1e-5, scale=8.0, alpha=2.0):
    return {"architecture": "Dokulorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "postln_alpha": alpha, "layers": layers}


CONFIGS = {
    # unlike layers in an order of their own
    "mixed": config(192, 500, [parallel(attention(6, 2, 40, 24, 16), state(3, 24, 40, (0.9, 0.999, 0.5)), 136),
                               retention(3, 32, 48, (0.97, 0.995, 0.8), ff=72),
                               parallel(attention(4, 4, 16, 56, 16, base=500.0, softcap=5.0), state(2, 72, 16, (0.99, 0.7))),
                               retention(5, 16, 8, (0.9, 0.99, 0.999, 0.6, 0.95), rot_dims=6, base=300.0)], scale=5.0, alpha=2.5),
    # sizes no vector load or tensor tile divides
    "odd": config(100, 301, [retention(3, 10, 13, (0.9, 0.99, 0.4), rot_dims=4, ff=33),
                             parallel(attention(3, 1, 14, 9, 6), state(5, 7, 11, (0.99, 0.9, 0.8, 0.7, 0.6)), 77),
                             parallel(attention(2, 2, 9, 5, 2), state(1, 3, 5, (0.95,)))], eps=1e-3, scale=1.0, alpha=1.0),
    # one of everything; a state that keeps all and one that keeps nothing
    "one": config(64, 70, [retention(1, 8, 8, (1.0,), base=3.0), parallel(attention(1, 1, 8, 8, 8), state(1, 8, 8, (0.0,)), 8)], scale=0.5, alpha=0.75),
    # nothing turns in some layers, the right mixer's sizes equal the left's
    "unrotated": config(72, 90, [retention(2, 16, 16, (0.99, 0.9), rot_dims=0), parallel(attention(2, 1, 16, 16, 0), state(2, 16, 16, (0.99, 0.9)), 40)]),
    # a real layer's head sizes
    "wide": config(512, 1000, [retention(4, 128, 128, (0.97, 0.99, 0.995, 0.999), ff=1024),
                               parallel(attention(16, 4, 128, 128, 64), state(4, 128, 128, (0.9, 0.99, 0.995, 0.999)), 520)]),
    # head widths at the ends of the tensor kernels' ranges, many query heads per key head, groups wider than a warp
    "edges": config(336, 260, [parallel(attention(20, 1, 104, 200, 48), state(2, 256, 256, (0.99, 0.9)), 96),
                               retention(2, 200, 256, (0.98, 0.999), rot_dims=128), parallel(attention(3, 3, 256, 72, 256), state(7, 136, 120, (0.9,) * 7))]),
    # past what the tensor kernels take
    "beyond": config(96, 80, [retention(1, 264, 264, (0.99,)), parallel(attention(2, 1, 24, 272, 8), state(1, 312, 40, (0.97,)), 24)]),
}


def tensors(cfg):
    """name -> shape, in the artifact's layout."""
    D, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}

    def heads(p, m, kv):
        out[p + "q"] = (m["heads"] * m["dim"], D)
        out[p + "k"] = (kv * m["dim"], D)
        out[p + "v"] = (kv * m["vdim"], D)
        out[p + "g"] = (m["heads"] * m["vdim"], D)
        out[p + "o"] = (D, m["heads"] * m["vdim"])

    for i, ly in enumerate(cfg["layers"]):
        l, m = "l%d." % i, ly["mixer"]
        out[l + "norm1"] = (D,)
        if ly["type"] == "retention":
            heads(l + "mix.", m, m["heads"])
        else:
            heads(l + "mix.left.", m["left"], m["left"]["kv_heads"])
            out[l + "mix.left.sink"] = (m["left"]["heads"],)
            heads(l + "mix.right.", m["right"], m["right"]["heads"])
            out[l + "mix.right.norm"] = (m["right"]["heads"] * m["right"]["vdim"],)
            out[l + "mix.left.out"] = out[l + "mix.right.out"] = (D,)
        if ly["mlp"] is not None:
            F = ly["mlp"]["ff"]
            out[l + "norm2"] = (D,)
            out[l + "mlp.gate"], out[l + "mlp.up"], out[l + "mlp.down"] = (F, D), (F, D), (D, F)
    out["final.norm"] = (D,)
    return out


def weights(cfg, seed):
    """Random bf16-valued weights."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensors(cfg).items():
        w = rng.standard_normal(shape)
        if len(shape) == 2:
            w /= np.sqrt(shape[1])
            if name == "embed":
                w *= np.sqrt(shape[1]) / cfg["embedding"]["scale"]  # the scaled rows have entries of size one
        elif name.endswith("sink"):
            w = 1.0 + w
        elif name.endswith("right.norm") or name.endswith(".out"):
            w = 1.0 + 0.4 * w
        else:
            w = 0.4 * w
        W[name] = bf16_round(w.astype(np.float32))
    return W
