"""Mubopel models end to end -- sessions, prompt passes, portions, decoding, verify blocks, generation, trace replay -- against
the float64 restatement."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from tests import latent_oracle as o
from tests.conftest import ROOT, synth_module
from tests.latent_models import model

pytestmark = pytest.mark.gpu

NAMES = ["mixed", "odd", "big", "huge", "wide_vocab"]
F32_TOL = 2e-5                                  # rms error of a position's logits over the rms of all logits


class Case:
    """A model, a token stream, the restatement's logits, and how far bf16 rounding alone moves them."""

    def __init__(self, name, n, seed=17):
        self.name = name
        self.shape, self.w, self.path = model(name)
        self.toks = synth_module().prompt_ids(n, self.shape.vocab, seed=seed)
        self.want = o.forward(self.shape.config(), self.w, self.toks)
        self.scale = float(np.sqrt(np.square(self.want).mean()))
        r = self.errors(o.forward(self.shape.config(), self.w, self.toks, rnd=o.to_bf16))
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


@pytest.fixture(scope="module", params=NAMES)
def case(request):
    return Case(request.param, {"mixed": 420, "odd": 300, "big": 200, "huge": 150, "wide_vocab": 90}[request.param])


def run(s, toks, cuts):
    """all logits of toks fed in portions of the given sizes (the last size repeats)"""
    rows, pos, i = [], 0, 0
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
            if case.name in ("big", "wide_vocab") and cuts in ([2], [5, 3, 2]):
                continue
            case.check(run(s, case.toks, cuts), dtype, what=cuts)      # the session's rows are used again from position 0 each time


def test_a_planted_mistake_would_show(case):
    cfg = case.shape.config()
    limit = max(case.tol["bfloat16"], 0.02)
    assert case.errors(o.forward(cfg, case.w, case.toks, sink=False)).max() > 2 * limit
    if any(l.kv_from is not None for l in case.shape.layers):
        assert case.errors(o.forward(cfg, case.w, case.toks, shared=False)).max() > 2 * limit


def test_rows_used_again_leave_nothing_behind(lg, case):
    other = synth_module().prompt_ids(len(case.toks), case.shape.vocab, seed=99)
    m = 70
    with lg.Session(case.path, None, len(case.toks) + 3) as s:
        fresh = run(s, case.toks[:m], [m])
    with lg.Session(case.path, None, len(case.toks) + 3) as s:
        run(s, other, [50, 1, 128])                            # a longer request first, in other portions
        assert np.array_equal(run(s, case.toks[:m], [m]), fresh)


def test_verify_rows_equal_plain_steps(lg, case):
    toks = case.toks
    base = 61                                                   # the block straddles a key tile
    with lg.Session(case.path, None, len(toks) + 3) as s:
        s.prefill(toks[:base])
        plain = np.stack([s.forward(int(toks[base + i]), base + i) for i in range(8)])
        succ = plain.argmax(axis=1)
        for M in (2, 5, 8):
            s.L.lgs_set_mtp_n(s.h, M); s.mtp_n = M
            adv, out = s.spec(toks[base:base + M], base)
            assert np.array_equal(out, succ[:M])
            want_adv = 1
            while want_adv < M and succ[want_adv - 1] == toks[base + want_adv]:
                want_adv += 1
            assert adv == want_adv
            assert np.array_equal(s.prefill_logits(toks[base:base + M], base, range(M)), plain[:M])


@pytest.mark.parametrize("name", ["mixed", "odd"])
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
    clear = top2[:, 1] - top2[:, 0] > 1e-4 * np.abs(want).max()
    assert clear.mean() > 0.95 and np.array_equal(want.argmax(axis=1)[clear], host[clear])
    # served precision: the same tokens wherever the margin is clear, teacher-forced on this stream
    with lg.Session(path, None, len(stream) + 8) as s:
        got = s.prefill_logits(stream[:-1], 0, range(len(prompt) - 1, len(stream) - 1))
        plain, _ = s.generate_device(prompt, 60)
        spec, st = s.generate_device(prompt, 60, 2, synth_module().replay_drafts(plain, shape.vocab, 0.6))
    clear = top2[:, 1] - top2[:, 0] > 0.3 * np.sqrt(np.square(want).mean())
    assert clear.any() and np.array_equal(got.argmax(axis=1)[clear], want.argmax(axis=1)[clear])
    assert np.array_equal(plain, spec) and 0 < st[1] < st[0]       # drafts were accepted and rejected; the stream is the plain one


def test_long_decoding(lg):
    c = Case("mixed", 1300, seed=8)
    with lg.Session(c.path, None, 1300) as s:
        c.check(run(s, c.toks, [700, 1]), "bfloat16")             # 600 single steps across nine key tiles


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompts_longer_than_a_block(lg, dtype):
    c = Case("mixed", 2310, seed=12)
    places = np.unique(np.concatenate([np.arange(0, 2310, 13), np.arange(2040, 2060), [2309]]))       # around the border of two blocks
    with lg.Session(c.path, None, 2400, dtype=dtype) as s:
        c.check(s.prefill_logits(c.toks, 0, places), dtype, places)
        # a portion that starts inside a block and a last stretch of a few tokens
        s.prefill(c.toks[:250], 0)
        c.check(s.prefill_logits(c.toks[250:2303], 250, places[places > 250][:150] - 250), dtype, places[places > 250][:150])
        c.check(s.prefill_logits(c.toks[2303:], 2303, range(7)), dtype, slice(2303, 2310))


def test_prefix_rows_and_embedding_rows(lg):
    c = Case("mixed", 120, seed=21)
    toks = c.toks
    with lg.Session(c.path, None, 200) as s:
        c.check(run(s, toks, [100, 1]), "bfloat16")
        s.save_prefix(64)
        run(s, synth_module().prompt_ids(120, c.shape.vocab, seed=22), [120])
        s.restore_prefix(64)
        b = np.concatenate([s.prefill_logits(toks[64:100], 64, range(36))] + [s.prefill_logits(toks[i:i + 1], i, [0]) for i in range(100, 120)])
        c.check(b, "bfloat16", slice(64, 120))
        k, v = s.kv_row(0, 5, 4096)
        assert np.array_equal(k, v) and np.abs(k).max() > 0
        # positions given as embedding rows instead of ids
        rows = np.random.default_rng(2).standard_normal((30, c.shape.width)).astype(np.float32)
        s.prefill_embd(rows, 0)
        got = s.prefill_logits(toks[:1], 30, [0])
        want = o.forward(c.shape.config(), c.w, None, embeddings=np.concatenate([rows, c.w["embed"][toks[:1]]]))
        assert np.sqrt(np.square(got - want[30]).mean()) / c.scale < c.tol["bfloat16"]


def test_out_of_range_requests_are_refused(lg):
    shape, w, path = model("odd")
    with lg.Session(path, None, 64) as s:
        for toks, pos, want in (([1, 2], 63, [0]), ([1, shape.vocab], 0, [1]), ([1], 0, [1]), ([-1], 0, [0])):
            with pytest.raises(ValueError):
                s.prefill_logits(toks, pos, want)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(lg, tmp_path, dtype):
    path = model("odd")[2]
    ca, cb = Case("odd", 80, seed=1), Case("odd", 25, seed=2)
    a, b, wa, wb = ca.toks, cb.toks, ca.want, cb.want
    steps, expect, n = [], {}, 0
    for name, toks, full, cuts in (("x", a, wa, [40, 2, 30, 1, 1, 6]), ("y", b, wb, [25])):
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
