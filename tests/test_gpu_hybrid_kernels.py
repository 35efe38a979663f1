"""Each mechanism of the state-space / windowed-attention design alone, through the kernel-level entry points, against its float64
restatement."""
import numpy as np
import pytest

from tests import hybrid_oracle as o

pytestmark = pytest.mark.gpu


def bf(x):
    return o.to_bf16(np.asarray(x, dtype=np.float32)).astype(np.float32)


def rel(got, want):
    return float(np.abs(got - want).max() / np.abs(want).max())


@pytest.mark.parametrize("m,m_up,k", [(48, 64, 64), (40, 51, 100), (272, 8, 23), (900, 2000, 1088)])
@pytest.mark.parametrize("n", [1, 3, 8, 9, 130, 300])
def test_paired_projections(lg, m, m_up, k, n):
    rng = np.random.default_rng(m + k + n)
    w, u, x, xu = (bf(rng.standard_normal(s) * a) for s, a in (((m, k), k ** -0.5), ((m_up, k), k ** -0.5), ((n, k), 1.0), ((n, k), 1.0)))
    f = [a.astype(np.float64) for a in (w, u, x, xu)]
    want, act = f[2] @ f[0].T, np.maximum(f[3] @ f[1].T, 0) ** 2
    for f32, tol, tol_a in ((False, 2e-5, 5e-3), (True, 2e-6, 4e-6)):
        got, ga = lg.dense_pair(w, u, x, xu, f32=f32)
        assert rel(got, want) < tol and rel(ga, act) < tol_a


def test_paired_projections_do_not_depend_on_the_block_width(lg):
    rng = np.random.default_rng(3)
    w, u, x, xu = (bf(rng.standard_normal(s)) for s in ((400, 700), (300, 700), (8, 700), (8, 700)))
    a8, b8 = lg.dense_pair(w, u, x, xu)
    for n in (1, 2, 5):
        a, b = lg.dense_pair(w, u, x[:n], xu[:n])
        assert np.array_equal(a, a8[:n]) and np.array_equal(b, b8[:n])


@pytest.mark.parametrize("n", [33, 64, 100, 2050, 4096, 7000, 16384])
def test_two_norms_of_one_sum(lg, n):
    rng = np.random.default_rng(n)
    f = lambda a: a.astype(np.float32).astype(np.float64)
    x, add, bias, w1, w2 = (f(rng.standard_normal(s) * c) for s, c in (((5, n), 1.0), ((5, n), 3.0), (n, 2.0), (n, 0.2), (n, 0.2)))
    eps = 0.05                                                          # large enough that its place inside the root shows
    for a, b in ((add, bias), (add, None), (None, bias), (None, None)):
        want = x + (0 if a is None else a) + (0 if b is None else b)
        gx, y1, y2 = lg.row_norm_pair(x, 1 + w1, 1 + w2, eps, a, b, f32=True)
        assert rel(gx, want) < 1e-6 and rel(y1, o.offset_norm(want, w1, eps)) < 2e-6 and rel(y2, o.offset_norm(want, w2, eps)) < 2e-6
    gx, y1, y2 = lg.row_norm_pair(x, 1 + w1, 1 + w2, eps, add)
    assert rel(y1, o.offset_norm(x + add, w1, eps)) < 5e-3 and rel(y2, o.offset_norm(x + add, w2, eps)) < 5e-3


# ---- state-space mixer ----------------------------------------------------------------------

SSM = [dict(heads=1, vdim=16, state=16, groups=1, norm_groups=1, taps=1), dict(heads=3, vdim=10, state=7, groups=1, norm_groups=5, taps=2),
       dict(heads=6, vdim=48, state=70, groups=3, norm_groups=2, taps=4), dict(heads=4, vdim=64, state=128, groups=2, norm_groups=4, taps=3),
       dict(heads=2, vdim=144, state=250, groups=1, norm_groups=3, taps=9), dict(heads=8, vdim=32, state=32, groups=8, norm_groups=8, taps=16)]


class Ssm:
    """A state-space mixer on random projected rows."""

    def __init__(self, lg, n, seed, **p):
        rng = np.random.default_rng(seed)
        self.lg, self.p, self.n = lg, p, n
        H, vd, N, G = p["heads"], p["vdim"], p["state"], p["groups"]
        self.inner, ch = H * vd, H * vd + 2 * G * N
        self.layer = lg.PlanLayer(mixer=lg.MIX_SSM, heads=H, vdim=vd, taps=p["taps"], state=N, groups=G, norm_groups=p["norm_groups"])
        f = lambda a: np.asarray(a, dtype=np.float32)
        self.w = [bf(rng.standard_normal((ch, p["taps"])) * p["taps"] ** -0.5 + np.eye(1, p["taps"], p["taps"] - 1)), bf(0.3 * rng.standard_normal(ch)),
                  f(np.log(np.expm1(np.exp(rng.uniform(np.log(0.01), np.log(0.6), H))))), f(np.log(rng.uniform(0.02, 3.0, H))), f(rng.standard_normal(H)),
                  f(1 + 0.2 * rng.standard_normal(self.inner))]
        self.rows = np.concatenate([bf(rng.standard_normal((n, self.inner + ch))), f(0.7 * rng.standard_normal((n, H)))], axis=1)
        self.eps = 0.02

    def want(self, rnd=o.exact, reset=()):
        p = self.p
        H, vd, N, G = p["heads"], p["vdim"], p["state"], p["groups"]
        conv, cb, dtb, A, D, norm = (a.astype(np.float64) for a in self.w)
        out, cuts = [], [0, *reset, self.n]
        for a, b in zip(cuts, cuts[1:]):
            r = self.rows[a:b].astype(np.float64)
            u = rnd(o.silu(o.short_conv(r[:, self.inner:-H], conv, cb)))
            x, B, Cm = np.split(u, [self.inner, self.inner + G * N], axis=1)
            y, _ = o.state_space(x.reshape(-1, H, vd), B.reshape(-1, G, N), Cm.reshape(-1, G, N), o.softplus(r[:, -H:] + dtb), A, D)
            out.append(o.gated_group_norm(y.reshape(len(r), -1), r[:, :self.inner], norm, p["norm_groups"], self.eps))
        return np.concatenate(out)

    def run(self, blocks, **kw):
        return self.lg.mixer_blocks(self.layer, self.w, self.rows, blocks, self.eps, max_seq=max(self.n, 64), **kw)

    def close(self, got, want, f32):
        d = np.abs(got - want).max(axis=1) / np.abs(want).max()
        assert d.max() < (2e-5 if f32 else 0.012), (float(d.max()), int(d.argmax()))


def cut(n, sizes):
    blocks, pos, i = [], 0, 0
    while pos < n:
        m = min(sizes[min(i, len(sizes) - 1)], n - pos)
        blocks.append((pos, m))
        pos, i = pos + m, i + 1
    return blocks


@pytest.mark.parametrize("p", SSM, ids=lambda p: "x".join(map(str, p.values())))
def test_state_space_in_portions(lg, p):
    n = 300
    c = Ssm(lg, n, 7, **p)
    want = {True: c.want(), False: c.want(o.to_bf16)}
    for sizes in ([n], [1], [2], [8], [9], [127, 1, 1, 130, 2], [128, 129], [5, 140, 3, 3, 64]):
        for f32 in (True, False):
            c.close(c.run(cut(n, sizes), f32=f32), want[f32], f32)
    c.close(c.run(cut(n, [64, 200, 7]), plain=True), want[False], False)
    # what a lost state would cost
    lost = c.want(reset=(150,))
    assert np.abs(lost[150:152] - want[True][150:152]).max() > 0.05 * np.abs(want[True]).max()


@pytest.mark.parametrize("p", SSM[1:4], ids=lambda p: "x".join(map(str, p.values())))
def test_state_space_steps_taken_back(lg, p):
    """Blocks cut back to any of their tokens, repeated, and wide blocks behind a narrow one that was cut back."""
    n = 200
    c = Ssm(lg, n, 8, **p)
    blocks = [(0, 40), (40, 8), (43, 8), (43, 8), (44, 1), (45, 5), (45, 5), (50, 8), (50, 3), (51, 100), (151, 2), (152, 1), (152, 8), (160, 8), (168, 32)]
    for f32 in (True, False):
        c.close(c.run(blocks, f32=f32), c.want(o.exact if f32 else o.to_bf16), f32)
        # a sequence that starts again where another one was
        got = c.run([(0, 100), (0, 5), (5, 60), (65, 1), (66, 134)], f32=f32)
        c.close(got, c.want(o.exact if f32 else o.to_bf16), f32)
    single = c.run(cut(n, [1]))
    for m in (2, 5, 8):
        assert np.array_equal(c.run(cut(n, [m])), single)              # bit for bit: verify rows are plain rows


def test_state_space_remembers_and_forgets(lg):
    """One token with a large step among small ones: its trace is still there hundreds of tokens later, and a strong decay wipes it."""
    p = dict(heads=2, vdim=16, state=16, groups=1, norm_groups=1, taps=2)
    c = Ssm(lg, 900, 9, **p)
    c.w[3] = np.log(np.array([0.002, 40.0], dtype=np.float32))
    c.rows[:, -2:] = -3.0
    c.rows[5, -2:] = 6.0
    c.rows[700, -1] = 12.0                                               # exp(-40 * 12): nothing is left of head 1's state
    want, other = c.want(), None
    saved = c.rows[5, -2:].copy()
    c.rows[5, -2:] = -3.0
    other = c.want()
    c.rows[5, -2:] = saved
    assert np.abs(want - other)[800].max() > 0.02 * np.abs(want).max()
    for sizes in ([900], [500, 300, 1], [100, 4]):
        c.close(c.run(cut(900, sizes), f32=True), want, True)
        c.close(c.run(cut(900, sizes)), c.want(o.to_bf16), False)


# ---- windowed attention mixer -----------------------------------------------------------------

ATT = [dict(heads=2, kv_heads=1, dim=16, vdim=16, window=64, taps=1), dict(heads=5, kv_heads=5, dim=9, vdim=13, window=10, taps=2),
       dict(heads=6, kv_heads=2, dim=48, vdim=96, window=100, taps=3), dict(heads=4, kv_heads=2, dim=64, vdim=128, window=129, taps=4),
       dict(heads=12, kv_heads=1, dim=32, vdim=48, window=0, taps=3), dict(heads=3, kv_heads=3, dim=100, vdim=112, window=1, taps=7),
       dict(heads=2, kv_heads=1, dim=40, vdim=200, window=65, taps=2)]


class Att:
    def __init__(self, lg, n, seed, maps=2, diff=0.35, gain=1.0, **p):
        rng = np.random.default_rng(seed)
        self.lg, self.p, self.n, self.maps, self.diff = lg, p, n, maps, diff
        H, G, d, vd, taps = p["heads"], p["kv_heads"], p["dim"], p["vdim"], p["taps"]
        self.scale = gain * d ** -0.5
        self.layer = lg.PlanLayer(mixer=lg.MIX_GROUPED, heads=H, kv_heads=G, dim=d, vdim=vd, maps=maps, window=p["window"], taps=taps, diff=diff, scale=self.scale)
        self.ch = [H * maps * d, G * maps * d, G * vd]
        self.w = [bf(rng.standard_normal((c, taps)) * 0.3 * taps ** -0.5 + np.eye(1, taps, taps - 1)) for c in self.ch]
        self.w += [bf(0.4 * rng.standard_normal(d)) for _ in range(4)]
        self.rows = bf(rng.standard_normal((n, sum(self.ch))))
        self.eps = 0.01

    def plant(self, i, key, h, m):
        """query i of head h, map m meets key `key` alone: one strong score (the filters must be a single tap of 1)"""
        H, G, d = self.p["heads"], self.p["kv_heads"], self.p["dim"]
        g = h // (H // G)
        v = np.random.default_rng(i * 7 + key).standard_normal(d)
        q0, k0 = (h * self.maps + m) * d, self.ch[0] + (g * self.maps + m) * d
        self.rows[key, k0:k0 + d] = bf(v)
        self.rows[i, q0:q0 + d] = bf(v * 12.0 / (self.scale * np.dot(v, v)))

    def want(self, rnd=o.exact, window=None):
        p, r = self.p, self.rows.astype(np.float64)
        H, G, d, vd = p["heads"], p["kv_heads"], p["dim"], p["vdim"]
        ws = [w.astype(np.float64) for w in self.w]
        q, k, v = (rnd(o.short_conv(u, w)) for u, w in zip(np.split(r, np.cumsum(self.ch)[:2], axis=1), ws))
        size = p["window"] if window is None else window
        q, k, v = q.reshape(-1, H, self.maps, d), k.reshape(-1, G, self.maps, d), v.reshape(-1, G, vd)
        if self.maps == 1:
            return o.attention_map(q[:, :, 0], k[:, :, 0], v, self.scale, 0, size).reshape(len(r), -1)
        return o.diff_attention(q, k, v, self.scale, 0, size, o.lam_of(*ws[3:], self.diff), self.diff, self.eps).reshape(len(r), -1)

    def run(self, blocks, max_seq=0, **kw):
        return self.lg.mixer_blocks(self.layer, self.w, self.rows, blocks, self.eps, max_seq=max_seq or self.n, **kw)

    def close(self, got, want, f32):
        d = np.abs(got - want).max(axis=1) / np.abs(want).max()
        assert d.max() < (5e-5 if f32 else 0.015), (float(d.max()), int(d.argmax()))


@pytest.mark.parametrize("p", ATT, ids=lambda p: "x".join(map(str, p.values())))
@pytest.mark.parametrize("maps", [2, 1])
def test_windowed_attention_in_portions(lg, p, maps):
    n = 330
    c = Att(lg, n, 11, maps=maps, **p)
    want = {True: c.want(), False: c.want(o.to_bf16)}
    for sizes in ([n], [1], [2], [8], [9], [63, 1, 1, 130, 2], [128, 129], [5, 140, 3, 3, 64]):
        for f32 in (True, False):
            c.close(c.run(cut(n, sizes), f32=f32), want[f32], f32)
    c.close(c.run(cut(n, [64, 200, 7]), plain=True), want[False], False)


@pytest.mark.parametrize("window", [1, 40, 63, 64, 65, 128, 191])
def test_keys_at_the_edges(lg, window):
    """Strong keys just inside and just outside of the window, at the borders of key tiles and blocks, and the first ones."""
    p = dict(heads=4, kv_heads=2, dim=32, vdim=48, window=window, taps=1)
    n, places = 420, [0, 1, window - 1, window, window + 1, 63, 64, 65, 127, 128, 129, 191, 192, 255, 256, 300, 383, 384, 419]
    for inside in (True, False):
        c = Att(lg, n, 13 + window, gain=3.0, **p)
        c.w[0][:], c.w[1][:] = 1.0, 1.0
        for j, i in enumerate(sorted({x for x in places if x < n})):
            key = i - window + (1 if inside else 0)
            if key >= 0:
                c.plant(i, key, j % 4, (j // 4) % 2)
        want = c.want(o.to_bf16)
        exact = c.want()
        for sizes in ([n], [1], [200, 1], [60, 5, 3, 300, 2], [128, 64, 65, 8]):
            c.close(c.run(cut(n, sizes)), want, False)
        c.close(c.run(cut(n, [100, 1, 7, 250, 2]), f32=True), exact, True)
        # a window that is one token off would be far outside of the tolerance
        off = c.want(window=window + (-1 if inside and window > 1 else 1))
        assert np.abs(off - exact).max() > 0.2 * np.abs(exact).max()


def test_far_key_among_hundreds(lg):
    p = dict(heads=4, kv_heads=1, dim=32, vdim=32, window=900, taps=1)
    c = Att(lg, 1000, 17, gain=2.0, **p)
    c.w[0][:], c.w[1][:] = 1.0, 1.0
    for j, (i, key) in enumerate([(999, 100), (998, 99), (950, 640), (900, 1), (899, 0), (640, 3), (997, 128)]):
        c.plant(i, key, j % 4, j % 2)
    want, exact = c.want(o.to_bf16), c.want()
    for sizes in ([1000], [890, 1], [500, 300, 3]):
        c.close(c.run(cut(1000, sizes)), want, False)
    c.close(c.run(cut(1000, [980, 1]), f32=True), exact, True)


def test_attention_blocks_taken_back_and_started_again(lg):
    c = Att(lg, 260, 19, **ATT[2])
    blocks = [(0, 60), (60, 8), (63, 8), (63, 8), (64, 1), (65, 5), (70, 100), (170, 8), (175, 8), (183, 77)]
    again = [(0, 200), (0, 5), (5, 130), (135, 1), (136, 124)]
    for f32 in (True, False):
        want = c.want(o.exact if f32 else o.to_bf16)
        c.close(c.run(blocks, f32=f32), want, f32)
        c.close(c.run(again, f32=f32), want, f32)
    single = c.run(cut(260, [1]))
    for m in (2, 5, 8):
        assert np.array_equal(c.run(cut(260, [m])), single)


def test_ring_of_cache_rows_wraps(lg):
    """A window much smaller than the sequence: rows are overwritten, by narrow and by wide blocks."""
    p = dict(heads=2, kv_heads=1, dim=16, vdim=16, window=100, taps=2)
    n = 5200                                                             # the ring holds 2304 rows
    c = Att(lg, n, 23, **p)
    want = c.want(o.to_bf16)
    for sizes in ([2048, 2040, 300, 8, 1, 1, 1, 800], [700, 2048, 2048, 5], [1500]):
        c.close(c.run(cut(n, sizes)), want, False)


def test_scores_that_grow_along_the_keys(lg):
    """Every tile raises the running maximum, so outputs are rescaled throughout."""
    p = dict(heads=2, kv_heads=1, dim=16, vdim=96, window=0, taps=1)
    c = Att(lg, 400, 29, **p)
    c.w[0][:], c.w[1][:] = 1.0, 1.0
    c.rows[:, :c.ch[0]] = 0
    c.rows[:, 0:c.ch[0]:16] = 4.0 / c.scale
    k0 = c.ch[0]
    c.rows[:, k0] = bf(np.linspace(-20, 30, 400)); c.rows[:, k0 + 16] = bf(np.linspace(-5, 60, 400))
    for sizes in ([400], [200, 1], [3]):
        c.close(c.run(cut(400, sizes)), c.want(o.to_bf16), False)
    c.close(c.run([(0, 400)], f32=True), c.want(), True)


def test_sizes_out_of_range_are_refused(lg):
    c = Ssm(lg, 20, 1, **SSM[0])
    for blocks in ([(0, 21)], [(-1, 4)], [(0, 0)]):
        with pytest.raises(ValueError):
            c.run(blocks)
    big = Ssm(lg, 9, 1, heads=1, vdim=16, state=300, groups=1, norm_groups=1, taps=2)
    with pytest.raises(ValueError):
        big.run([(0, 9)])
