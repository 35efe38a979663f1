"""Each mechanism of the latent-attention design alone, through the kernel-level entry points, against its float64 restatement."""
import numpy as np
import pytest

from tests import latent_oracle as o

pytestmark = pytest.mark.gpu


def bf(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32)


def rel(got, want):
    return float(np.abs(got - want).max() / np.abs(want).max())


@pytest.mark.parametrize("m,k", [(48, 64), (40, 100), (272, 23), (2000, 1088), (8, 9), (320, 4096)])
@pytest.mark.parametrize("n", [1, 3, 8, 9, 130, 300])
def test_dense_matmul(lg, m, k, n):
    rng = np.random.default_rng(m * 7 + k + n)
    w, u, x = (bf(rng.standard_normal(s) * a) for s, a in (((m, k), k ** -0.5), ((m, k), k ** -0.5), ((n, k), 1.0)))
    plain = x.astype(np.float64) @ w.T.astype(np.float64)
    gated = np.maximum(plain, 0) * (x.astype(np.float64) @ u.T.astype(np.float64))
    assert rel(lg.dense_matmul(w, x), plain) < 2e-5
    assert rel(lg.dense_matmul(w, x, f32=True), plain) < 2e-6
    assert rel(lg.dense_matmul(w, x, u), gated) < 5e-3                  # the gated epilogue rounds to bf16
    assert rel(lg.dense_matmul(w, x, u, f32=True), gated) < 2e-6


def test_dense_matmul_rows_do_not_depend_on_the_block_width(lg):
    rng = np.random.default_rng(3)
    w, x = bf(rng.standard_normal((400, 700))), bf(rng.standard_normal((8, 700)))
    all8 = lg.dense_matmul(w, x)
    for n in (1, 2, 5):
        assert np.array_equal(lg.dense_matmul(w, x[:n]), all8[:n])


@pytest.mark.parametrize("n", [33, 64, 100, 320, 2050, 4096, 7000, 16384])
@pytest.mark.parametrize("center", [True, False])
def test_row_norm_with_residual(lg, n, center):
    rng = np.random.default_rng(n)
    x, add = rng.standard_normal((5, n)) + 0.3, rng.standard_normal((5, n)) * 4 - 1
    w, aw = 1 + 0.2 * rng.standard_normal(n), 1 + 0.2 * rng.standard_normal(n)
    norm = o.layer_norm if center else o.rms_norm
    eps = 0.05                                                          # large enough that its place inside the root shows
    f = lambda a: a.astype(np.float32).astype(np.float64)
    x, add, w, aw = map(f, (x, add, w, aw))
    want_x = x + 0.3 * norm(add, aw, eps)
    gx, gy = lg.row_norm(x, w, eps, add, aw, 0.3, center, f32=True)
    assert rel(gx, want_x) < 1e-6 and rel(gy, norm(want_x, w, eps)) < 2e-6
    gx, gy = lg.row_norm(x, w, eps, center=center)
    assert np.array_equal(gx, x.astype(np.float32)) and rel(gy, norm(x, w, eps)) < 5e-3


def _latent_case(rng, n, H, kv, rot, pos, planted=()):
    """Queries and latent rows; `planted` positions hold a key that one query of some head matches strongly."""
    q = rng.standard_normal((n, H, kv + rot)) * 0.15
    c = rng.standard_normal((pos + n, kv + rot))
    for j, key in enumerate(planted):
        h = j % H
        i = n - 1 if key <= pos else key - pos
        d = rng.standard_normal(kv + rot)
        c[key] = d
        q[i, h] = d * 20.0 / np.dot(d, d)
    return bf(q), bf(c)


def _latent_want(q, c, sink, kv, pos, scale):
    q, c = q.astype(np.float64), c.astype(np.float64)
    n, H, d = q.shape
    k = np.repeat(c[:, None, :kv], H, axis=1)
    return o.attention(q[..., :kv], q[..., kv:], k, c[:, kv:], k, sink.astype(np.float64), scale, pos)


EDGES = (0, 1, 63, 64, 65, 127, 128, 191)


@pytest.mark.parametrize("H,kv,rot", [(1, 16, 4), (5, 37, 6), (16, 128, 32), (20, 512, 64), (40, 250, 64), (3, 560, 16)])
@pytest.mark.parametrize("n,pos", [(1, 0), (2, 0), (1, 63), (1, 64), (3, 62), (8, 125), (1, 1000), (5, 2047)])
def test_latent_attention_over_the_cache(lg, H, kv, rot, n, pos):
    rng = np.random.default_rng(H + kv + n + pos)
    planted = [p for p in EDGES + (pos - 64, pos - 1, pos) if 0 <= p < pos + n]
    q, c = _latent_case(rng, n, H, kv, rot, pos, planted)
    sink = (0.5 + rng.standard_normal(H)).astype(np.float32)
    want = _latent_want(q, c, sink, kv, pos, 1.0)
    scale_of = np.abs(want).max()
    for form, f32, tol in ((0, False, 6e-3), (1, False, 6e-3), (1, True, 2e-5)):
        if form == 0 and kv > 512:
            continue
        got = lg.latent_attn(q, c, sink, kv, pos, 1.0, max_seq=4096 if pos < 100 else 0, rows_form=bool(form), f32=f32)
        assert np.abs(got - want).max() / scale_of < tol, (form, f32)
    # a mask that is off by one would be far outside of the tolerance
    if pos > 0 and n == 1:
        off = _latent_want(q, c[:-1], sink, kv, pos - 1, 1.0)
        assert np.abs(off - want).max() / scale_of > 0.02


def test_latent_rows_do_not_depend_on_the_block_width(lg):
    rng = np.random.default_rng(9)
    H, kv, rot, pos = 20, 128, 32, 300
    q, c = _latent_case(rng, 8, H, kv, rot, pos)
    sink = np.ones(H, np.float32)
    all8 = lg.latent_attn(q, c, sink, kv, pos, 1.0, max_seq=1024)
    for n in (1, 3, 4):
        assert np.array_equal(lg.latent_attn(q[:n], c[:pos + n], sink, kv, pos, 1.0, max_seq=1024), all8[:n])
    for i in (2, 7):                                                    # a later row on its own
        assert np.array_equal(lg.latent_attn(q[i:i + 1], c[:pos + i + 1], sink, kv, pos + i, 1.0, max_seq=1024), all8[i:i + 1])


@pytest.mark.parametrize("H,dim,rot,vd", [(1, 16, 16, 16), (3, 20, 6, 12), (4, 128, 64, 128), (2, 48, 80, 200), (2, 192, 64, 256), (5, 64, 16, 96)])
@pytest.mark.parametrize("n,pos", [(9, 0), (64, 0), (65, 63), (129, 0), (200, 500), (130, 1023), (17, 64)])
def test_prompt_attention(lg, H, dim, rot, vd, n, pos):
    rng = np.random.default_rng(H + dim + n + pos)
    q, k = rng.standard_normal((n, H, dim + rot)) * 0.2, rng.standard_normal((pos + n, H, dim))
    kr, v = rng.standard_normal((pos + n, rot)), rng.standard_normal((pos + n, H, vd))
    gate, sink = rng.standard_normal((n, H, vd)), (0.5 + rng.standard_normal(H)).astype(np.float32)
    # one strong key per chosen query: the first ones, tile borders, just inside the causal edge and far away
    for j, (i, key) in enumerate([(n - 1, 0), (n - 1, pos), (n // 2, pos + n // 2), (n // 2, 63), (n - 2, 64), (8, 1), (n - 1, pos + n - 1), (0, pos)]):
        if key <= pos + i:
            h, d = j % H, rng.standard_normal(dim + rot)
            q[i, h] = d * 25.0 / np.dot(d, d)
            k[key, h] = d[:dim]
            kr[key] = d[dim:]
    # scores that grow along the keys make every tile raise the running maximum
    q[3 % n, 0] = 0.0
    q[3 % n, 0, 0] = 1.0
    k[:, 0, 0] = np.linspace(-40, 60, pos + n)
    q, k, kr, v = map(bf, (q, k, kr, v))
    f = [a.astype(np.float64) for a in (q, k, kr, v)]
    att = o.attention(f[0][..., :dim], f[0][..., dim:], f[1], f[2], f[3], sink.astype(np.float64), 1.0, pos)
    want = att * o.sigmoid(gate.astype(np.float32).astype(np.float64))
    got = lg.latent_prompt_attn(q, k, kr, v, gate, sink, pos, 1.0)
    assert np.abs(got - want).max() / np.abs(want).max() < 6e-3


@pytest.mark.parametrize("pos", [0, 5, 62, 63, 64, 300])
def test_sink_takes_its_share_once(lg, pos):
    """Sinks that hold about half of the weight: leaving one out, scaling it or counting it per tile would show."""
    rng = np.random.default_rng(pos)
    H, d, rot, n = 6, 48, 16, 12
    scale = 0.25                                                        # not applied to the sink
    q, c, v = bf(rng.standard_normal((n, H, d + rot)) * 0.3), bf(rng.standard_normal((pos + n, d + rot))), bf(rng.standard_normal((pos + n, H, d)))
    sink = (np.log(pos + n) + rng.standard_normal(H)).astype(np.float32)
    want = _latent_want(q, c, sink, d, pos, scale)
    lost = _latent_want(q, c, sink - 1e9, d, pos, scale)
    assert np.abs(lost - want).max() > 0.1 * np.abs(want).max()
    for form, f32 in ((False, False), (True, False), (True, True)):
        got = lg.latent_attn(q[:8], c[:pos + 8], sink, d, pos, scale, rows_form=form, f32=f32)
        assert np.abs(got - want[:8]).max() < (2e-5 if f32 else 6e-3) * np.abs(want).max()
    f = [x.astype(np.float64) for x in (q, c, v)]
    k = np.repeat(f[1][:, None, :d], H, axis=1)
    gate = np.full((n, H, d), 0.3)
    want = o.attention(f[0][..., :d], f[0][..., d:], k, f[1][:, d:], f[2], sink.astype(np.float64), scale, pos) * o.sigmoid(0.3)
    got = lg.latent_prompt_attn(q, k, c[:, d:], v, gate, sink, pos, scale)
    assert np.abs(got - want).max() < 6e-3 * np.abs(want).max()
