"""Baporax models end to end -- sessions, prompt passes, portions, decoding, verify blocks, generation, prefixes, trace replay -- against
the float64 restatement."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from tests import hybrid_oracle as o
from tests.conftest import ROOT, synth_module
from tests.hybrid_models import model

pytestmark = pytest.mark.gpu

F32_TOL = 4e-5                                  # rms error of a position's logits over the rms of all logits
LENGTH = {"looped": 400, "odd": 260, "big": 330, "huge": 150, "states": 120, "windows": 300}


class Case:
    """A model, a token stream, the restatement's logits, and how far bf16 rounding alone moves them."""

    def __init__(self, name, n, seed=17):
        self.name = name
        self.shape, self.w, self.path = model(name)
        self.toks = synth_module().prompt_ids(n, self.shape.vocab, seed=seed)
        self.cfg = self.shape.config()
        self.want = o.forward(self.cfg, self.w, self.toks)
        self.scale = float(np.sqrt(np.square(self.want).mean()))
        r = self.errors(o.forward(self.cfg, self.w, self.toks, rnd=o.to_bf16))
        self.tol = {"float32": F32_TOL, "bfloat16": 3 * float(r.max())}
        self.mid = {"float32": F32_TOL, "bfloat16": 1.5 * float(np.median(r))}

    def errors(self, got, rows=slice(None)):
        """per position: rms error over the vocabulary, over the rms of all expected logits"""
        return np.sqrt(np.square(got - self.want[rows]).mean(axis=1)) / self.scale

    def check(self, got, dtype, rows=slice(None), what=""):
        e = self.errors(got, rows)
        assert e.max() < self.tol[dtype], (what, e.max(), self.tol[dtype])
        if len(e) > 20:
            assert np.median(e) < self.mid[dtype], (what, np.median(e), self.mid[dtype])


@pytest.fixture(scope="module", params=sorted(LENGTH))
def case(request):
    return Case(request.param, LENGTH[request.param])


def run(s, toks, cuts, pos=0):
    """all logits of toks fed in portions of the given sizes (the last size repeats)"""
    rows, i = [], 0
    while pos < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - pos)
        rows.append(s.prefill_logits(toks[pos:pos + n], pos, range(n)))
        pos += n
        i += 1
    return np.concatenate(rows)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_and_single_tokens(lg, case, dtype):
    n = len(case.toks)
    with lg.Session(case.path, None, n + 3, dtype=dtype) as s:
        for cuts in ([n], [1], [2], [5, 3, 2], [9, 8, 17, 2, 64, 1, 1, 130], [n - 40, 1]):
            if case.name in ("big", "states") and cuts in ([2], [5, 3, 2]):
                continue
            case.check(run(s, case.toks, cuts), dtype, what=cuts)      # every sequence starts over at position 0


def test_planted_mistakes_would_show(case):
    limit = max(case.tol["bfloat16"], 0.02)
    kinds = {l.type for l in case.shape.layers}
    if "attention" in kinds:
        assert case.errors(o.forward(case.cfg, case.w, case.toks, window_shift=1)).max() > limit
    lost = case.errors(o.forward(case.cfg, case.w, case.toks, forget=60))
    assert "mamba2" not in kinds or lost.max() > limit
    assert not case.shape.loop or case.errors(o.forward(case.cfg, case.w, case.toks, steps=False)).max() > limit


def test_sequences_leave_nothing_behind(lg, case):
    other = synth_module().prompt_ids(len(case.toks), case.shape.vocab, seed=99)
    m = 70
    with lg.Session(case.path, None, len(case.toks) + 3) as s:
        fresh = run(s, case.toks[:m], [m])
        steps = run(s, case.toks[:20], [1])
    with lg.Session(case.path, None, len(case.toks) + 3) as s:
        run(s, other, [50, 1, 128])                            # a longer request first, in other portions
        assert np.array_equal(run(s, case.toks[:m], [m]), fresh)
        run(s, other[:33], [33])
        assert np.array_equal(run(s, case.toks[:20], [1]), steps)


def test_verify_rows_equal_plain_steps(lg, case):
    toks = case.toks
    base = 61                                                   # the block straddles a key tile
    with lg.Session(case.path, None, len(toks) + 3) as s:
        s.prefill(toks[:base])
        plain = np.stack([s.forward(int(toks[base + i]), base + i) for i in range(8)])
        succ = plain.argmax(axis=1)
        for M in (2, 5, 8):
            s.prefill(toks[:base])                              # (the states have moved on)
            s.L.lgs_set_mtp_n(s.h, M); s.mtp_n = M
            adv, out = s.spec(toks[base:base + M], base)
            assert np.array_equal(out, succ[:M])
            want_adv = 1
            while want_adv < M and succ[want_adv - 1] == toks[base + want_adv]:
                want_adv += 1
            assert adv == want_adv
            assert np.array_equal(s.prefill_logits(toks[base:base + M], base, range(M)), plain[:M])       # the same block again
            # cut back to every one of its tokens and continued
            for keep in range(1, M + 1):
                s.prefill_logits(toks[base:base + M], base, [])
                if keep < 8:
                    assert np.array_equal(s.forward(int(toks[base + keep]), base + keep), plain[keep])
                s.prefill(toks[:base])


def test_prompts_through_many_resident_kernels(lg):
    c = Case("deep", 400, seed=3)
    with lg.Session(c.path, None, 420) as s:
        first = run(s, c.toks, [400])
        c.check(first, "bfloat16")
        for _ in range(20):
            s.prefill(c.toks[:100])
            assert np.array_equal(run(s, c.toks, [400]), first)


def test_positions_without_state_are_refused(lg):
    c = Case("looped", 80)
    with lg.Session(c.path, None, 200) as s:
        s.prefill(c.toks[:50])
        for pos in (10, 49, 51, 120):
            with pytest.raises(ValueError):
                s.prefill_logits(c.toks[:3], pos, [0])
        c.check(s.prefill_logits(c.toks[50:], 50, range(30)), "bfloat16", slice(50, 80))
        for toks, pos, want in (([1, 2], 199, [0]), ([1, c.shape.vocab], 0, [1]), ([1], 0, [1]), ([-1], 0, [0])):
            with pytest.raises(ValueError):
                s.prefill_logits(toks, pos, want)


@pytest.mark.parametrize("name", ["looped", "odd", "windows"])
def test_greedy_generation_follows_the_restatement(lg, name):
    shape, w, path = model(name)
    prompt = list(synth_module().prompt_ids(75, shape.vocab, seed=4))
    n_gen = 150
    with lg.Session(path, None, 75 + n_gen + 24, dtype="float32") as s:
        host, _ = s.generate(prompt, n_gen)
        dev, _ = s.generate_device(prompt, n_gen)
        hidden = s.last_hidden()
    assert np.array_equal(host, dev) and len(host) == n_gen and np.isfinite(hidden).all()
    stream = np.array(prompt + list(map(int, host)))
    want = o.forward(shape.config(), w, stream[:-1])[len(prompt) - 1:]
    top2 = np.sort(want, axis=1)[:, -2:]
    clear = top2[:, 1] - top2[:, 0] > 3e-4 * np.abs(want).max()
    assert clear.mean() > 0.95 and np.array_equal(want.argmax(axis=1)[clear], host[clear])
    # served precision: the same tokens wherever the margin is clear, teacher-forced on this stream
    with lg.Session(path, None, len(stream) + 24) as s:
        got = s.prefill_logits(stream[:-1], 0, range(len(prompt) - 1, len(stream) - 1))
        plain, _ = s.generate_device(prompt, 60)
        spec, st = s.generate_device(prompt, 60, 2, synth_module().replay_drafts(plain, shape.vocab, 0.6))
        blocking, _ = s.generate(prompt, 60, 2, synth_module().replay_drafts(plain, shape.vocab, 0.6))
    clear = top2[:, 1] - top2[:, 0] > 0.3 * np.sqrt(np.square(want).mean())
    assert clear.any() and np.array_equal(got.argmax(axis=1)[clear], want.argmax(axis=1)[clear])
    assert np.array_equal(plain, spec) and 0 < st[1] < st[0]       # drafts were accepted and rejected; the stream is the plain one
    assert np.array_equal(blocking[:60], plain[:60])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(lg, dtype):
    c = Case("looped", 1300, seed=8)
    with lg.Session(c.path, None, 1300, dtype=dtype) as s:
        c.check(run(s, c.toks, [700, 1]), dtype)             # 600 single steps


@pytest.fixture(scope="module")
def long_case():
    return Case("looped", 4700, seed=12)                         # the windowed layers' rows wrap


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompts_longer_than_a_block(lg, long_case, dtype):
    c = long_case
    n = len(c.toks)
    places = np.unique(np.concatenate([np.arange(0, n, 31), np.arange(2040, 2060), np.arange(4090, 4110), [n - 1]]))       # around the borders of blocks
    with lg.Session(c.path, None, n, dtype=dtype) as s:
        c.check(s.prefill_logits(c.toks, 0, places), dtype, places)
        # a portion that starts inside a block and a last stretch of a few tokens
        s.prefill(c.toks[:250], 0)
        some = places[(places >= 250) & (places < n - 7)]
        c.check(s.prefill_logits(c.toks[250:n - 7], 250, some - 250), dtype, some)
        c.check(s.prefill_logits(c.toks[n - 7:], n - 7, range(7)), dtype, slice(n - 7, n))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefix_state_and_embedding_rows(lg, dtype):
    c = Case("looped", 160, seed=21)
    toks = c.toks
    with lg.Session(c.path, None, 200, dtype=dtype) as s:
        s.prefill(toks[:100])
        s.save_prefix(100)
        a = run(s, toks, [30, 1], pos=100)
        run(s, synth_module().prompt_ids(120, c.shape.vocab, seed=22), [120])
        s.restore_prefix(100)
        assert np.array_equal(run(s, toks, [30, 1], pos=100), a)
        c.check(a, dtype, slice(100, 160))
        k, v = s.kv_row(1, 5, 4096)                              # the second layer run is attention, the first has no rows
        assert np.array_equal(k, v) and np.abs(k).max() > 0 and s.kv_row(0, 5, 4096)[0] is None
        # positions given as embedding rows instead of ids
        rows = np.random.default_rng(2).standard_normal((30, c.shape.width)).astype(np.float32)
        s.prefill_embd(rows, 0)
        got = s.prefill_logits(toks[:1], 30, [0])
        want = o.forward(c.cfg, c.w, None, embeddings=np.concatenate([rows, c.w["embed"][toks[:1]]]))
        assert np.sqrt(np.square(got - want[30]).mean()) / c.scale < c.tol[dtype]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(lg, tmp_path, dtype):
    path = model("odd")[2]
    ca, cb = Case("odd", 80, seed=1), Case("odd", 25, seed=2)
    steps, expect, n = [], {}, 0
    for name, toks, full, cuts in (("x", ca.toks, ca.want, [40, 2, 30, 1, 1, 6]), ("y", cb.toks, cb.want, [25])):
        pos = 0
        for c in cuts:
            want = [] if c == 30 else [c - 1] if c < 3 else [c - 1, 0, c // 2]
            steps.append({"step": n, "entries": [{"id": name, "tokens": [int(t) for t in toks[pos:pos + c]], "want": want}],
                          "end": [name] if pos + c == len(toks) else []})
            if want:
                expect[n] = full[[pos + j for j in want]]
            pos += c
            n += 1
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "80"],
                       input="".join(json.dumps(x) + "\n" for x in steps), capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr[-500:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(n)]
    for i in range(n):
        f = tmp_path / f"{i}.f32"
        assert f.exists() == (i in expect)
        if i in expect:
            got = np.fromfile(f, "<f4").reshape(expect[i].shape)
            assert np.sqrt(np.square(got - expect[i]).mean(axis=1)).max() / ca.scale < ca.tol[dtype]


@pytest.mark.parametrize("family,name", [("hybrid", "big"), ("hybrid", "looped"), ("hybrid", "deep"), ("latent", "mixed"), ("latent", "big")])
def test_bits_do_not_depend_on_what_the_caches_hold(lg, family, name):
    """Prompts and steps behind an overwritten L2: copies and code arrive late and in another order, the bits stay."""
    import torch
    from tests import latent_models
    shape, _, path = model(name) if family == "hybrid" else latent_models.model(name)
    toks = synth_module().prompt_ids(330, shape.vocab, seed=31)
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    with lg.Session(path, None, 340) as s:
        want = run(s, toks, [320, 1])
        for k in range(60):
            flush.zero_()
            torch.cuda.synchronize()
            got = s.prefill_logits(toks[:320], 0, range(320))
            assert np.array_equal(got, want[:320]), int(np.flatnonzero((got != want[:320]).any(axis=1))[0])
            if k % 10 == 0:
                for i in range(320, 330):
                    flush.zero_()
                    torch.cuda.synchronize()
                    assert np.array_equal(s.prefill_logits(toks[i:i + 1], i, [0]), want[i:i + 1])
