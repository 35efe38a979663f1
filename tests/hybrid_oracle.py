"""Plain, slow float64 restatement of the Baporax design (state-space layers and windowed differential attention, looped), one
function per mechanism, for tests.

A model is its config.json as a dict and its tensors as float arrays under their checkpoint names.  Nothing is cached, cut or
batched: forward() runs a whole sequence, token by token where a layer is a recurrence, and returns the logits of every position.
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


def unit(x, eps):
    """x over its root mean square along the last axis"""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def offset_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from 1"""
    return unit(x, eps) * (1.0 + w)


def silu(z):
    return z * 0.5 * (1.0 + np.tanh(0.5 * z))


def softplus(z):
    return np.logaddexp(0.0, z)


def short_conv(u, w, bias=None):
    """Causal convolution over time, channel by channel: u [tokens, channels], w [channels, taps], the last tap on the present."""
    out = np.zeros_like(u)
    taps = w.shape[1]
    for back in range(min(taps, len(u))):
        out[back:] += u[:len(u) - back] * w[:, taps - 1 - back]
    return out if bias is None else out + bias


def state_space(x, B, C, dt, A_log, D):
    """x [n, heads, vdim], B and C [n, groups, N], dt [n, heads] (positive): y [n, heads, vdim] and the last state."""
    n, H, vd = x.shape
    G = B.shape[1]
    of = np.arange(H) // (H // G)
    S = np.zeros((H, vd, B.shape[2]))
    y = np.empty_like(x)
    for t in range(n):
        S = S * np.exp(-np.exp(A_log) * dt[t])[:, None, None] + (dt[t][:, None] * x[t])[:, :, None] * B[t][of][:, None, :]
        y[t] = np.einsum("hvn,hn->hv", S, C[t][of]) + D[:, None] * x[t]
    return y, S


def gated_group_norm(y, z, w, groups, eps):
    """gate first, then every one of `groups` equal parts over its own root mean square"""
    g = y * silu(z)
    return unit(g.reshape(len(g), groups, -1), eps).reshape(g.shape) * w


def window_mask(n_queries, n_keys, first, size):
    """[queries, keys]: query i sits at position first + i and sees the last `size` positions up to its own (0: all of them)"""
    back = first + np.arange(n_queries)[:, None] - np.arange(n_keys)[None, :]
    return (back >= 0) & ((back < size) if size else True)


def softmax(scores, seen):
    s = np.where(seen, scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def attention_map(q, k, v, scale, first, size):
    """q [n, H, d], k [keys, G, d], v [keys, G, vd] -> [n, H, vd]; head h reads group h // (H / G)"""
    of = np.arange(q.shape[1]) // (q.shape[1] // k.shape[1])
    out = []
    for i in range(0, len(q), 256):                  # (keys that no query of the stretch sees are left out)
        some = q[i:i + 256]
        lo, hi = max(0, first + i - size + 1) if size else 0, min(len(k), first + i + len(some))
        s = np.einsum("nhd,khd->hnk", some, k[lo:hi, of], optimize=True) * scale
        out.append(np.einsum("hnk,khv->nhv", softmax(s, window_mask(len(some), hi - lo, first + i - lo, size)), v[lo:hi, of], optimize=True))
    return np.concatenate(out)


def differential(a1, a2, lam, diff, eps):
    return unit(a1 - lam * a2, eps) * (1.0 - diff)


def lam_of(lq1, lk1, lq2, lk2, diff):
    return np.exp(np.dot(lq1, lk1)) - np.exp(np.dot(lq2, lk2)) + diff


def diff_attention(q, k, v, scale, first, size, lam, diff, eps):
    """q [n, H, 2, d], k [keys, G, 2, d], v [keys, G, vd] -> [n, H, vd]"""
    a = [attention_map(q[:, :, m], k[:, :, m], v, scale, first, size) for m in range(2)]
    return differential(a[0], a[1], lam, diff, eps)


def mamba_mixer(w, p, m, h, eps, rnd=exact):
    H, vd, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * vd
    u = rnd(h @ w[p + "in"].T)
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], (h @ w[p + "in"].T)[:, 2 * inner + 2 * G * N:]
    c = rnd(silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"])))
    x, B, C = np.split(c, [inner, inner + G * N], axis=1)
    y, _ = state_space(x.reshape(-1, H, vd), B.reshape(-1, G, N), C.reshape(-1, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return rnd(gated_group_norm(rnd(y.reshape(-1, inner)), z, w[p + "norm"], m["norm_groups"], eps)) @ w[p + "o"].T


def attention_mixer(w, p, m, h, eps, rnd=exact, window=None):
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (rnd(short_conv(rnd(h @ w[p + t].T), w[p + t + ".conv"])) for t in "qkv")
    lam = lam_of(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
    size = m["mask"]["size"] if window is None else window
    o = diff_attention(q.reshape(-1, H, 2, d), k.reshape(-1, G, 2, d), v.reshape(-1, G, vd), m["scale"], 0, size, lam, m["diff"], eps)
    return rnd(o.reshape(len(h), -1)) @ w[p + "o"].T


def feed_forward(w, p, h, rnd=exact):
    return rnd(np.maximum(h @ w[p + "up"].T, 0.0) ** 2) @ w[p + "down"].T


def layer_runs(cfg):
    """(layer, number of the pass whose step comes before it or None) in the order of execution"""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, *, embeddings=None, rnd=exact, layers=None, window_shift=0, forget=None, steps=True):
    """Logits [tokens, vocab].  rnd is applied to what enters a product (with to_bf16 it shows how far rounding alone moves the
    logits).  Mistakes planted on purpose, to show that a comparison would notice: window_shift widens or narrows every window,
    forget = p loses the recurrent state and the convolutions' history at position p, steps False leaves out the loop's vectors.
    `layers`, if given, receives the residual rows after every layer run."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] if embeddings is None else np.asarray(embeddings, dtype=np.float64)
    for i, step in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if step is not None and steps:
            x = x + w["loop.step"][step]
        h = rnd(offset_norm(x, w[p + "norm1"], eps))
        if layer["type"] == "mamba2":
            parts = [h] if forget is None else [h[:forget], h[forget:]]
            add = np.concatenate([mamba_mixer(w, p + "mix.", layer["mixer"], part, eps, rnd) for part in parts if len(part)])
        else:
            size = layer["mixer"]["mask"]["size"]
            add = attention_mixer(w, p + "mix.", layer["mixer"], h, eps, rnd, size + window_shift)
        if layer["mlp"] is not None:
            add = add + feed_forward(w, p + "mlp.", rnd(offset_norm(x, w[p + "norm2"], eps)), rnd)
        x = x + add
        if layers is not None:
            layers.append(x)
    return rnd(offset_norm(x, w["final.norm"], eps)) @ w["embed"].T * cfg["logit_scale"]
