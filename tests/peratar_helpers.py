"""Small Peratar models with random weights for the tests: configuration, weights, artifact folder."""
import json
import os
import struct

import numpy as np


def bf16_bits(a):
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_round(a):
    return (bf16_bits(a).astype(np.uint32) << 16).view(np.float32)


def mixer(heads, dim, rot, vdim, rank, base=10000.0, rot_dims=None, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
         "scale": (dim + rot) ** -0.5 if scale is None else scale}
    if rot:
        m["rot"] = {"base": base, "dims": rot if rot_dims is None else rot_dims}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def layer(mix, ff):
    return {"type": "latent_attention", "mixer": mix, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, eps=1e-5, softcap=20.0):
    return {"architecture": "Peratar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": softcap,
            "layers": layers}


CONFIGS = {
    # unlike layers: other head counts over a shared cache, a layer without a feed-forward, two owners
    "mixed": config(192, 500, [layer(mixer(4, 24, 16, 40, 48), 200), layer(mixer(6, 40, 16, 16, 48, kv_from=0), None),
                               layer(mixer(3, 16, 8, 24, 72, base=500.0), 136), layer(mixer(5, 8, 8, 32, 72, base=500.0, kv_from=2), 72),
                               layer(mixer(2, 32, 16, 8, 48, kv_from=0), 64)]),
    # sizes no vector load or tensor tile divides
    "odd": config(100, 301, [layer(mixer(3, 10, 6, 13, 20), 77), layer(mixer(5, 7, 6, 9, 20, kv_from=0), 33),
                             layer(mixer(1, 12, 2, 5, 11), None)], eps=1e-3, softcap=5.0),
    # one of everything
    "one": config(64, 70, [layer(mixer(1, 8, 2, 8, 8, base=3.0), 8)], softcap=2.0),
    # no rotated part at all; only part of the rotated dimensions turn; the first layers have no feed-forward
    "unrotated": config(72, 90, [layer(mixer(2, 16, 0, 16, 24), None), layer(mixer(1, 8, 8, 8, 16), None),
                                 layer(mixer(3, 8, 16, 16, 24, rot_dims=6), 40)]),
    # a real layer's head sizes, more than sixteen heads
    "wide": config(512, 1000, [layer(mixer(20, 128, 64, 128, 512), 1024), layer(mixer(17, 128, 64, 128, 512, kv_from=0), 520)]),
    # latent and value widths at the ends of the tensor kernels' ranges
    "edges": config(320, 260, [layer(mixer(2, 56, 24, 256, 136), 96), layer(mixer(9, 104, 48, 200, 1024), 128)]),
}


def tensors(cfg):
    """name -> shape, in the artifact's layout."""
    D, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, ly in enumerate(cfg["layers"]):
        p, m = "l%d." % i, ly["mixer"]
        H = m["heads"]
        out[p + "norm1"] = (D,)
        out[p + "mix.q"] = (H * (m["dim"] + m["rot_dim"]), D)
        if m.get("kv_from") is None:
            out[p + "mix.dkv"] = (m["kv_rank"] + m["rot_dim"], D)
            out[p + "mix.dkv.norm"] = (m["kv_rank"],)
        out[p + "mix.uk"] = (H * m["dim"], m["kv_rank"])
        out[p + "mix.uv"] = (H * m["vdim"], m["kv_rank"])
        out[p + "mix.g"] = (H, D)
        out[p + "mix.o"] = (D, H * m["vdim"])
        out[p + "rg1"], out[p + "rg1.b"] = (D, D), (D,)
        if ly["mlp"] is not None:
            F = ly["mlp"]["ff"]
            out[p + "norm2"] = (D,)
            out[p + "mlp.up"], out[p + "mlp.up.b"] = (F, D), (F,)
            out[p + "mlp.down"], out[p + "mlp.down.b"] = (D, F), (D,)
            out[p + "mlp.act"] = (2,)
            out[p + "rg2"], out[p + "rg2.b"] = (D, D), (D,)
        out[p + "dwa"] = (i + 2,)
    out["final.norm"] = (D,)
    out["head"] = (cfg["vocab"], D)
    return out


def weights(cfg, seed, q_gain=2.0):
    """Random bf16-valued weights; q_gain sharpens the attention so that single keys stand out."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensors(cfg).items():
        if len(shape) == 2:
            w = rng.standard_normal(shape) / np.sqrt(shape[1])
            if name == "embed":
                w = rng.standard_normal(shape)
            if name.endswith(".q"):
                w *= q_gain
            if ".rg" in name:
                w *= 1.5
        elif "norm" in name:
            w = 1.0 + 0.4 * rng.standard_normal(shape)
        elif name.endswith("dwa"):
            w = 0.4 * rng.standard_normal(shape)
            w[-1] += 1.0
        else:
            w = 0.7 * rng.standard_normal(shape)
        W[name] = bf16_round(w.astype(np.float32))
    return W


def write_artifact(path, cfg, W, skew=0):
    """config.json + model.safetensors; skew shifts the data by odd bytes."""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blob = {}, b""
    for name, w in W.items():
        b = bf16_bits(w).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(w.shape), "data_offsets": [len(blob), len(blob) + len(b)]}
        blob += b
    h = json.dumps(head).encode()
    h += b" " * ((8 - len(h) % 8) % 8 + skew)
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + blob)
    return str(path)


def rel(got, want):
    """Root mean square difference over the want's root mean square."""
    want = np.asarray(want, np.float64)
    return float(np.sqrt(((np.asarray(got, np.float64) - want) ** 2).mean() / (want ** 2).mean()))
