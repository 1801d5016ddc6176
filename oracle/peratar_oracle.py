"""Plain restatement of the Peratar decoder in numpy, one function per mechanism.

What the tests hold csrc/decoder.cu and its kernels to: slow, whole sequence at once, float64 unless asked
otherwise, no cache and no batching.  It shares no code with the product path.  `W` is a dict from
tensor names to float arrays, `cfg` the parsed config.json.

Notation: x_t is row t of the stream, n the layer norm, m the mixer, f the feed-forward, X_j the
stream after layer j - 1 (X_0 = embedding), a_ij the averaging weights of layer i.
"""
import numpy as np


def sigmoid(z):
    z = np.asarray(z)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def softplus(z):
    return np.maximum(z, 0) + np.log1p(np.exp(-np.abs(z)))


def layer_norm(x, w, eps):
    """(x - mean) / sqrt(mean square deviation + eps) * w, over the last axis."""
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def rotate_pairs(x, pos, base, dims):
    """Neighbouring pairs (2i, 2i+1) of the first `dims` entries turn by pos * base^(-2i/dims);
    x [T, ..., >= dims], pos [T]."""
    out = x.copy()
    i = np.arange(dims // 2)
    ang = np.asarray(pos, np.float64)[:, None] * np.float64(base) ** (-2.0 * i / dims)
    shape = (len(pos),) + (1,) * (x.ndim - 2) + (dims // 2,)
    c, s = np.cos(ang).reshape(shape).astype(x.dtype), np.sin(ang).reshape(shape).astype(x.dtype)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def rotate_part(x, pos, mx):
    """The rotated part of a query or key under the mixer's own rotation (none when it is empty)."""
    return rotate_pairs(x, pos, mx["rot"]["base"], mx["rot"]["dims"]) if mx["rot_dim"] else x


def latent_kv(h, pos, w_dkv, w_norm, mx, eps):
    """-> (latent [T, kv_rank], shared rotated key part [T, rot_dim])."""
    y = h @ w_dkv.T
    r = mx["kv_rank"]
    return rms_norm(y[:, :r], w_norm, eps), rotate_part(y[:, r:], pos, mx)


def causal_softmax(s):
    """s [T, T] scores of one head; row i keeps columns 0..i."""
    T = s.shape[0]
    s = np.where(np.tril(np.ones((T, T), bool)), s, -np.inf)
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def latent_attention(h, c, kr, W, p, mx):
    """The mixer on input rows h, with the latent c and rotated key part kr of the layer that owns
    the cache; p is the tensor prefix of this layer's mixer."""
    H, d, r, v = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
    T = h.shape[0]
    pos = np.arange(T)
    q = (h @ W[p + "q"].T).reshape(T, H, d + r)
    qr = rotate_part(q[:, :, d:], pos, mx)
    k = (c @ W[p + "uk"].T).reshape(T, H, d)
    val = (c @ W[p + "uv"].T).reshape(T, H, v)
    gate = sigmoid(h @ W[p + "g"].T)
    out = np.empty((T, H, v), h.dtype)
    for a in range(H):
        s = (q[:, a, :d] @ k[:, a].T + qr[:, a] @ kr.T) * mx["scale"]
        out[:, a] = (causal_softmax(s) @ val[:, a]) * gate[:, a:a + 1]
    return out.reshape(T, H * v) @ W[p + "o"].T


def xielu(z, p, q):
    return np.where(z > 0, softplus(p) * z * z + 0.5 * z,
                    (0.5 + softplus(q)) * (np.expm1(np.minimum(z, 0)) - np.minimum(z, 0)) + 0.5 * z)


def feed_forward(h, W, p):
    u = h @ W[p + "up"].T + W[p + "up.b"]
    a = W[p + "act"]
    return xielu(u, a[0], a[1]) @ W[p + "down"].T + W[p + "down.b"]


def gated(y, h, w, b):
    """A sublayer's result under its residual gate, which reads the sublayer's input."""
    return y * sigmoid(h @ w.T + b)


def depth_average(streams, a):
    return sum(a[j] * streams[j] for j in range(len(streams)))


def soft_cap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


def forward(W, cfg, tokens, want_layers=False, dtype=np.float64):
    """-> logits [T, vocab] (and the averaged stream after every layer, [layers, T, width])."""
    W = {k: np.asarray(v, dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens, np.int64)]
    X, taps, kv = [x], [], {}
    pos = np.arange(len(tokens))
    for i, ly in enumerate(cfg["layers"]):
        l, mx = "l%d." % i, ly["mixer"]
        if mx.get("kv_from") is None:
            kv[i] = latent_kv(x, pos, W[l + "mix.dkv"], W[l + "mix.dkv.norm"], mx, eps)
            src = i
        else:
            src = mx["kv_from"]
        y = latent_attention(x, kv[src][0], kv[src][1], W, l + "mix.", mx)
        x = x + layer_norm(gated(y, x, W[l + "rg1"], W[l + "rg1.b"]), W[l + "norm1"], eps)
        if ly.get("mlp") is not None:
            y = feed_forward(x, W, l + "mlp.")
            x = x + layer_norm(gated(y, x, W[l + "rg2"], W[l + "rg2.b"]), W[l + "norm2"], eps)
        X.append(x)
        x = depth_average(X, W[l + "dwa"])
        taps.append(x)
    logits = soft_cap(layer_norm(x, W["final.norm"], eps) @ W["head"].T, cfg.get("logit_softcap"))
    return (logits, np.stack(taps)) if want_layers else logits


def greedy(W, cfg, prompt, n, dtype=np.float64):
    """n greedy tokens after the prompt (the lowest index wins ties), recomputed from scratch each time."""
    ids = list(int(t) for t in prompt)
    out = []
    for _ in range(n):
        t = int(np.argmax(forward(W, cfg, ids, dtype=dtype)[-1]))
        out.append(t)
        ids.append(t)
    return out
