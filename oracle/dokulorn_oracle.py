"""Plain restatement of the Dokulorn decoder in numpy, one function per mechanism.

What the tests hold csrc/decoder.cu and its kernels to: slow, whole sequence at once, float64 unless asked
otherwise, no cache and no batching.  It shares no code with the product path.  `W` is a dict from
tensor names to float arrays, `cfg` the parsed config.json.

Notation: x is the stream, z the input of a sublayer, a the residual weight, g the per-head decay of a
linear-attention state S.
"""
import numpy as np


def sigmoid(z):
    z = np.asarray(z)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    """x over its root mean square along the last axis, eps under the root."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm_plain(x, w, eps):
    return unit_rms(x, eps) * w


def norm_one_plus(x, w, eps):
    """A norm whose stored weight is the distance from one."""
    return unit_rms(x, eps) * (1 + w)


def residual(x, y, w, a, eps):
    """The stream after a sublayer with result y: a weighted sum, normed afterwards."""
    return norm_one_plus(a * x + y, w, eps)


def rotate_halves(x, pos, base, dims):
    """Entries (i, i + dims/2) of the first `dims` turn by pos * base^(-2i/dims); x [T, ..., >= dims], pos [T]."""
    half = dims // 2
    if half == 0:
        return x
    out = x.copy()
    ang = np.asarray(pos, np.float64)[:, None] * np.float64(base) ** (-2.0 * np.arange(half) / dims)
    shape = (len(pos),) + (1,) * (x.ndim - 2) + (half,)
    c, s = np.cos(ang).reshape(shape).astype(x.dtype), np.sin(ang).reshape(shape).astype(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def rotated(x, pos, mx):
    r = mx.get("rot")
    return rotate_halves(x, pos, r["base"], r["dims"]) if r else x


def decayed_state(q, k, v, g, S=None):
    """Linear attention of one head: S <- g S + k_t v_t^T, o_t = S^T q_t, token by token.
    q, k [T, dim], v [T, vdim] -> (o [T, vdim], S [dim, vdim])."""
    S = np.zeros((k.shape[1], v.shape[1]), v.dtype) if S is None else S
    o = np.empty_like(v)
    for t in range(len(q)):
        S = g * S + np.outer(k[t], v[t])
        o[t] = q[t] @ S
    return o, S


def heads_of(x, w, n):
    y = x @ w.T
    return y.reshape(len(x), n, -1)


def retention(z, W, p, mx, eps):
    """Rotated queries and keys over decayed states; every head's result over its own root mean square,
    a SiLU gate over all of them."""
    T, H = len(z), mx["heads"]
    pos = np.arange(T)
    q = rotated(heads_of(z, W[p + "q"], H), pos, mx)
    k = rotated(heads_of(z, W[p + "k"], H), pos, mx) * mx["dim"] ** -0.5
    v = heads_of(z, W[p + "v"], H)
    o = np.stack([decayed_state(q[:, h], k[:, h], v[:, h], mx["decay"][h])[0] for h in range(H)], 1)
    return (unit_rms(o, eps).reshape(T, -1) * silu(z @ W[p + "g"].T)) @ W[p + "o"].T


def sink_softmax(s, sink):
    """Causal weights of one head [T, T]; the denominator also holds exp(sink)."""
    T = len(s)
    s = np.where(np.tril(np.ones((T, T), bool)), s, -np.inf)
    m = np.maximum(s.max(-1, keepdims=True), sink)
    e = np.exp(s - m)
    return e / (e.sum(-1, keepdims=True) + np.exp(sink - m))


def soft_cap(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def grouped_attention(z, W, p, mx, eps):
    """Softmax attention of H query heads over G key/value heads: rotation, then unit norms of query and
    key, capped scores, a sink per head, a sigmoid gate on the result's elements."""
    T, H, G = len(z), mx["heads"], mx["kv_heads"]
    pos = np.arange(T)
    q = unit_rms(rotated(heads_of(z, W[p + "q"], H), pos, mx), eps)
    k = unit_rms(rotated(heads_of(z, W[p + "k"], G), pos, mx), eps)
    v = heads_of(z, W[p + "v"], G)
    out = np.empty((T, H, mx["vdim"]), z.dtype)
    for h in range(H):
        j = h // (H // G)
        s = soft_cap((q[:, h] @ k[:, j].T) * mx["scale"], mx.get("softcap"))
        out[:, h] = sink_softmax(s, W[p + "sink"][h]) @ v[:, j]
    return (out.reshape(T, -1) * sigmoid(z @ W[p + "g"].T)) @ W[p + "o"].T


def lightning(z, W, p, mx, eps):
    """Decayed states over SiLU-activated queries, keys and values; one plain norm over all heads, a sigmoid gate."""
    T, H = len(z), mx["heads"]
    q, k, v = (silu(heads_of(z, W[p + n], H)) for n in "qkv")
    o = np.stack([decayed_state(q[:, h], k[:, h], v[:, h], mx["decay"][h])[0] for h in range(H)], 1)
    return (norm_plain(o.reshape(T, -1), W[p + "norm"], eps) * sigmoid(z @ W[p + "g"].T)) @ W[p + "o"].T


def parallel(z, W, p, mx, eps):
    """Both mixers on the same input; the mean of their results, each normed over the width first."""
    a = norm_plain(grouped_attention(z, W, p + "left.", mx["left"], eps), W[p + "left.out"], eps)
    b = norm_plain(lightning(z, W, p + "right.", mx["right"], eps), W[p + "right.out"], eps)
    return 0.5 * (a + b)


MIXERS = {"retention": retention, "parallel": parallel}


def feed_forward(z, W, p):
    return (gelu_tanh(z @ W[p + "gate"].T) * (z @ W[p + "up"].T)) @ W[p + "down"].T


def forward(W, cfg, tokens, want_layers=False, dtype=np.float64):
    """-> logits [T, vocab] (and the stream after every layer, [layers, T, width])."""
    W = {k: np.asarray(v, dtype) for k, v in W.items()}
    eps, a = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = W["embed"][np.asarray(tokens, np.int64)] * dtype(cfg["embedding"]["scale"])
    taps = []
    for i, ly in enumerate(cfg["layers"]):
        l = "l%d." % i
        x = residual(x, MIXERS[ly["type"]](x, W, l + "mix.", ly["mixer"], eps), W[l + "norm1"], a, eps)
        if ly.get("mlp") is not None:
            x = residual(x, feed_forward(x, W, l + "mlp."), W[l + "norm2"], a, eps)
        taps.append(x)
    logits = norm_one_plus(x, W["final.norm"], eps) @ W["embed"].T
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
