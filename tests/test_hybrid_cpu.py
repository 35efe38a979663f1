"""Baporax checkpoint folders and layer runs without a GPU, and the float64 restatement's own identities."""
import ctypes as C
import json
import os

import numpy as np
import pytest

from tests import hybrid_oracle as o
from tests.conftest import synth_module
from tests.hybrid_models import model, shapes
from tests.test_checkpoint_cpu import lib  # noqa: F401  (fixture)


@pytest.fixture()
def plans(lib):  # noqa: F811
    lib.lg_plan_runs.argtypes = [C.c_void_p]
    lib.lg_plan_run_layer.argtypes = [C.c_void_p, C.c_int, C.POINTER(C.c_int)]
    return lib


@pytest.mark.parametrize("name", sorted(shapes()))
def test_plan_and_tensors_of_a_folder(plans, name):
    shape, w, path = model(name)
    g = plans.load_model(path.encode())
    assert g and plans.lg_plan_present(g)
    ptr = plans.lg_plan_read(g)
    p = ptr.contents
    assert (p.n_layer, p.width, p.vocab, p.norm_kind, p.act, p.form) == (len(shape.layers), shape.width, shape.vocab, 0, 1, 1)
    assert p.norm_eps == np.float32(shape.eps) and p.norm_offset == 1.0 and p.logit_scale == np.float32(shape.logit_scale)
    for i, l in enumerate(shape.layers):
        q = p.layer[i]
        assert (q.heads, q.vdim, q.taps, q.ff) == (l.heads, l.vdim, l.conv, l.ff)
        if l.type == "mamba2":
            assert (q.mixer, q.state, q.groups, q.norm_groups) == (3, l.state, l.groups, l.norm_groups)
        else:
            assert (q.mixer, q.kv_heads, q.dim, q.maps, q.window) == (2, l.kv_heads, l.dim, 2, l.window)
            assert q.scale == np.float32(l.mixer()["scale"]) and q.diff == np.float32(l.diff)
    runs = []
    for r in range(plans.lg_plan_runs(ptr)):
        step = C.c_int(-5)
        L = plans.lg_plan_run_layer(ptr, r, C.byref(step))
        runs.append((L, None if step.value < 0 else step.value))
    assert runs == o.layer_runs(shape.config()) and len(runs) == len(shape.runs())
    assert plans.gguf_find_tensor(g, b"blk.0.attn_norm.weight") and not plans.gguf_find_tensor(g, b"blk.0.post_attention_norm.weight")
    plans.lg_plan_free(ptr)
    plans.free_gguf(g)


def _folder(tmp_path, edit):
    s = synth_module()
    shape = shapes()["looped"]
    path = str(tmp_path / "m")
    s.write_checkpoint(path, shape, 1)
    cfg = shape.config()
    edit(cfg)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return path.encode()


@pytest.mark.parametrize("edit", [
    lambda c: c.pop("logit_scale"), lambda c: c.update(width="wide"), lambda c: c["layers"][0].update(type="latent_attention"),
    lambda c: c["layers"][0]["mixer"].pop("groups"), lambda c: c["layers"][1]["mixer"].pop("diff"), lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][1]["mlp"].update(kind="routed"), lambda c: c["loop"].pop("times"), lambda c: c["norm"].pop("eps")])
def test_unusable_configurations_are_refused(lib, tmp_path, edit):  # noqa: F811
    assert not lib.load_model(_folder(tmp_path, edit))


@pytest.mark.parametrize("edit", [
    lambda c: c["layers"][0]["mixer"].update(groups=3), lambda c: c["layers"][0]["mixer"].update(norm_groups=7), lambda c: c["layers"][0]["mixer"].update(conv=0),
    lambda c: c["layers"][1]["mixer"].update(kv_heads=3), lambda c: c["layers"][1]["mixer"].update(conv=17), lambda c: c["layers"][1]["mixer"].update(scale=0),
    lambda c: c["loop"].update(stop=9), lambda c: c["loop"].update(start=3), lambda c: c["loop"].update(times=-1)])
def test_unusable_plans_are_refused(lib, tmp_path, edit):  # noqa: F811
    g = lib.load_model(_folder(tmp_path, edit))
    assert g and not lib.lg_plan_read(g)
    lib.free_gguf(g)


def test_restatement_identities():
    shape, w, _ = model("looped")
    toks = synth_module().prompt_ids(90, shape.vocab, seed=3)
    a = o.forward(shape.config(), w, toks)
    assert np.allclose(a[:60], o.forward(shape.config(), w, toks[:60]), atol=1e-8)          # causal
    rng = np.random.default_rng(0)
    u = rng.standard_normal((12, 3))
    f = rng.standard_normal((3, 4))
    assert np.allclose(o.short_conv(u, f)[5], sum(f[:, j] * u[2 + j] for j in range(4)))
    assert np.allclose(o.short_conv(u, f)[1], f[:, 3] * u[1] + f[:, 2] * u[0])
    # a state that does not decay is a sum; the convolution form of the recurrence
    x, B, Cm, dt = rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 1, 5)), rng.standard_normal((9, 1, 5)), rng.uniform(0.1, 1, (9, 2))
    A = np.array([0.3, -1.0])
    y, S = o.state_space(x, B, Cm, dt, A, np.zeros(2))
    for h in range(2):
        run = np.cumsum(-np.exp(A[h]) * dt[:, h])
        P = np.tril((Cm[:, 0] @ B[:, 0].T) * np.exp(run[:, None] - run[None, :]) * dt[None, :, h])
        assert np.allclose(P @ x[:, h], y[:, h])
    seen = o.window_mask(4, 6, 2, 3)
    assert [list(np.flatnonzero(r)) for r in seen] == [[0, 1, 2], [1, 2, 3], [2, 3, 4], [3, 4, 5]]
    assert o.window_mask(2, 3, 1, 0).tolist() == [[True, True, False], [True, True, True]]
    z = rng.standard_normal((2, 6))
    g = o.gated_group_norm(z, np.full((2, 6), 50.0), np.ones(6), 3, 0.0)
    assert np.allclose(np.square(g.reshape(2, 3, 2)).mean(-1), 1.0)
