"""Plain, slow float64 restatement of the Mubopel design, one function per mechanism, for tests.

A model is its config.json as a dict and its tensors as float arrays under their checkpoint names.  Nothing is cached, cut or
batched: forward() runs a whole sequence and returns the logits of every position.
"""
import numpy as np


def widen(bits: np.ndarray) -> np.ndarray:
    """bf16 bit patterns -> float64"""
    return np.left_shift(bits.astype(np.uint32), 16).view(np.float32).astype(np.float64)


def to_bf16(x):
    """the values of x rounded to bf16"""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32).astype(np.float64)


def exact(x):
    return x


def layer_norm(x, w, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return w * d / np.sqrt(np.square(d).mean(axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return w * x / np.sqrt(np.square(x).mean(axis=-1, keepdims=True) + eps)


def rotate(x, positions, base, dims):
    """Pairs (2i, 2i + 1) of the first `dims` columns turn by position * base^(-2i/dims); x is [tokens, ..., columns]."""
    z = x[..., :dims:2] + 1j * x[..., 1:dims:2]
    turn = np.outer(positions, np.power(float(base), -np.arange(0, dims, 2) / dims))
    z = z * np.exp(1j * turn).reshape(turn.shape[:1] + (1,) * (x.ndim - 2) + turn.shape[1:])
    out = np.array(x, dtype=np.float64)
    out[..., :dims:2], out[..., 1:dims:2] = z.real, z.imag
    return out


def sink_softmax(scores, sink):
    """scores [heads, queries, keys] (-inf = not seen), sink [heads] or None: weights whose missing mass went to the sink."""
    top = scores.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink[:, None, None])
    e = np.exp(scores - top)
    total = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink[:, None, None] - top)
    return e / total


def causal(scores, first):
    """Query i of the block sits at position first + i and sees the keys up to it."""
    n, k = scores.shape[-2:]
    return np.where(np.arange(k)[None, :] <= first + np.arange(n)[:, None], scores, -np.inf)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def latent_rows(w, p, m, h, positions, eps, rnd=exact):
    """What a layer caches: the normed latent and the rotated key part."""
    r = h @ w[p + "dkv"].T
    return (rnd(rms_norm(r[:, :m["kv_rank"]], w[p + "dkv.norm"], eps)),
            rnd(rotate(r[:, m["kv_rank"]:], positions, m["rot"]["base"], m["rot"]["dims"])))


def queries(w, p, m, h, positions, eps, rnd=exact):
    c = rnd(rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps))
    q = (c @ w[p + "uq"].T).reshape(len(h), m["heads"], m["dim"] + m["rot_dim"])
    return rnd(q[..., :m["dim"]]), rnd(rotate(q[..., m["dim"]:], positions, m["rot"]["base"], m["rot"]["dims"]))


def attention(q, q_rot, k, k_rot, v, sink, scale, first=0):
    """q [n, H, d], q_rot [n, H, r], k [keys, H, d], k_rot [keys, r], v [keys, H, vd] -> [n, H, vd]"""
    s = np.einsum("nhd,khd->hnk", q, k) + np.einsum("nhr,kr->hnk", q_rot, k_rot)
    return np.einsum("hnk,khv->nhv", sink_softmax(causal(s * scale, first), sink), v)


def latent_attention(w, p, m, h, rows, positions, eps, sink=True, rnd=exact):
    c, k_rot = rows
    H = m["heads"]
    q, q_rot = queries(w, p, m, h, positions, eps, rnd)
    k = rnd((c @ w[p + "uk"].T).reshape(len(c), H, m["dim"]))
    v = rnd((c @ w[p + "uv"].T).reshape(len(c), H, m["vdim"]))
    o = attention(q, q_rot, k, k_rot, v, w[p + "sink"] if sink else None, m["scale"])
    return rnd(o.reshape(len(h), -1) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def feed_forward(w, p, h, rnd=exact):
    return rnd(np.maximum(h @ w[p + "gate"].T, 0.0) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg, w, tokens, *, sink=True, shared=True, embeddings=None, rnd=exact):
    """Logits [tokens, vocab].  sink / shared False: mistakes planted on purpose (no sink; a borrowing layer makes rows of its
    own from the lender's weights), to show that a comparison would notice.  rnd is applied to what enters a product (and to the
    cached rows): with to_bf16 it shows how far rounding alone moves the logits."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][np.asarray(tokens)] if embeddings is None else np.asarray(embeddings, dtype=np.float64)
    positions = np.arange(len(x))
    cache = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rnd(layer_norm(x, w[p + "norm1"], eps))
        src = m.get("kv_from", i)
        if src == i:
            cache[i] = latent_rows(w, p + "mix.", m, h, positions, eps, rnd)
        rows = cache[src] if shared else latent_rows(w, f"l{src}.mix.", m, h, positions, eps, rnd)
        x = x + mult * layer_norm(latent_attention(w, p + "mix.", m, h, rows, positions, eps, sink, rnd), w[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            h = rnd(layer_norm(x, w[p + "norm2"], eps))
            x = x + mult * layer_norm(feed_forward(w, p + "mlp.", h, rnd), w[p + "norm2b"], eps)
    return rnd(layer_norm(x, w["final.norm"], eps)) @ w["embed"].T
