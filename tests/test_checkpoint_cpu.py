"""Checkpoint folders and layer plans without a GPU: what the readers accept, what they refuse, and the float64 restatement's own
identities."""
import ctypes as C
import json
import os

import numpy as np
import pytest

from tests import latent_oracle as o
from tests.conftest import lg_module, synth_module
from tests.latent_models import model, shapes


class Plan(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("n_layer", "width", "vocab", "norm_kind", "act")] + \
               [("norm_eps", C.c_float), ("residual_mult", C.c_float), ("layer", C.POINTER(lg_module().PlanLayer)), ("form", C.c_int),
                ("norm_offset", C.c_float), ("logit_scale", C.c_float)] + [(n, C.c_int) for n in ("loop_start", "loop_stop", "loop_times")]


class Tensor(C.Structure):
    _fields_ = [("name", C.c_char_p), ("n_dims", C.c_uint32), ("dims", C.c_uint64 * 4), ("type", C.c_uint32), ("offset", C.c_uint64), ("data", C.c_void_p)]


@pytest.fixture(scope="module")
def lib(lg):
    L = lg.load()
    L.load_model.restype = C.c_void_p; L.load_model.argtypes = [C.c_char_p]
    L.free_gguf.argtypes = [C.c_void_p]
    L.lg_plan_read.restype = C.POINTER(Plan); L.lg_plan_read.argtypes = [C.c_void_p]
    L.lg_plan_free.argtypes = [C.POINTER(Plan)]
    L.lg_plan_present.argtypes = [C.c_void_p]
    L.gguf_find_tensor.restype = C.POINTER(Tensor); L.gguf_find_tensor.argtypes = [C.c_void_p, C.c_char_p]
    return L


@pytest.mark.parametrize("name", sorted(shapes()))
def test_plan_and_tensors_of_a_folder(lib, name):
    shape, w, path = model(name)
    g = lib.load_model(path.encode())
    assert g and lib.lg_plan_present(g)
    p = lib.lg_plan_read(g).contents
    assert (p.n_layer, p.width, p.vocab, p.norm_kind) == (len(shape.layers), shape.width, shape.vocab, 1)
    assert p.norm_eps == np.float32(shape.eps) and p.residual_mult == np.float32(shape.residual_mult)
    for i, l in enumerate(shape.layers):
        q = p.layer[i]
        assert (q.heads, q.dim, q.rot_dim, q.vdim, q.q_rank, q.kv_rank, q.ff, q.rot_dims) == \
               (l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.ff, l.rot_dim)
        assert q.kv_src == (i if l.kv_from is None else l.kv_from)
        assert q.scale == np.float32(l.score_scale()) and q.rot_base == np.float32(l.base)
    t = lib.gguf_find_tensor(g, b"blk.0.attn_q_b.weight").contents
    l = shape.layers[0]
    assert list(t.dims)[:2] == [l.q_rank, l.heads * (l.dim + l.rot_dim)] and t.type == 30
    raw = np.ctypeslib.as_array(C.cast(t.data, C.POINTER(C.c_uint8)), (t.dims[0] * t.dims[1] * 2,)).copy().view(np.uint16)
    assert np.array_equal(o.widen(raw).reshape(t.dims[1], t.dims[0]), w["l0.mix.uq"])
    assert not lib.gguf_find_tensor(g, b"blk.99.attn_norm.weight")
    lib.lg_plan_free(C.pointer(p))
    lib.free_gguf(g)


def _folder(tmp_path, edit=None, tensors=None):
    s = synth_module()
    shape = shapes()["odd"]
    path = str(tmp_path / "m")
    s.write_checkpoint(path, shape, 1)
    cfg = shape.config()
    if edit:
        edit(cfg)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(cfg, f)
    if tensors:
        tensors(os.path.join(path, "model.safetensors"))
    return path.encode()


@pytest.mark.parametrize("edit", [
    lambda c: c.update(architecture="Nobody"), lambda c: c.pop("width"), lambda c: c.update(vocab=1.5), lambda c: c.update(layers=[]),
    lambda c: c["layers"][1].update(type="recurrence"), lambda c: c["layers"][0]["mixer"].pop("heads"),
    lambda c: c["layers"][0]["mlp"].update(kind="routed"), lambda c: c["norm"].pop("eps")])
def test_unusable_configurations_are_refused(lib, tmp_path, edit):
    assert not lib.load_model(_folder(tmp_path, edit))


@pytest.mark.parametrize("edit", [
    lambda c: c["layers"][0]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(kv_from=1),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8), lambda c: c["layers"][0]["mixer"].update(scale=0)])
def test_unusable_plans_are_refused(lib, tmp_path, edit):
    g = lib.load_model(_folder(tmp_path, edit))
    assert g and not lib.lg_plan_read(g)
    lib.free_gguf(g)


def test_damaged_files_are_refused(lib, tmp_path):
    def cut(f): os.truncate(f, os.path.getsize(f) - 2)
    def junk(f): open(f, "wb").write(b"\xff" * 64)
    def short(f): os.truncate(f, 6)
    for i, t in enumerate((cut, junk, short)):
        assert not lib.load_model(_folder(tmp_path / str(i), tensors=t))
    p = _folder(tmp_path / "x")
    open(os.path.join(p.decode(), "config.json"), "w").write('{"architecture": "Mubopel", ')
    assert not lib.load_model(p)
    assert not lib.load_model(str(tmp_path / "nowhere").encode())


def test_restatement_is_causal_and_rotations_keep_distances():
    shape, w, _ = model("mixed")
    toks = synth_module().prompt_ids(40, shape.vocab, seed=3)
    a = o.forward(shape.config(), w, toks)
    b = o.forward(shape.config(), w, toks[:25])
    assert np.allclose(a[:25], b, atol=1e-9)
    x = np.random.default_rng(0).standard_normal((6, 2, 8))
    y = o.rotate(x, np.arange(6), 100.0, 6)
    assert np.allclose(y[0], x[0]) and np.allclose(y[..., 6:], x[..., 6:]) and np.allclose(np.square(y).sum(-1), np.square(x).sum(-1))
    # a pair's product depends on the distance of the positions only
    z = o.rotate(np.repeat(x[:1], 6, axis=0), np.arange(6) + 11, 100.0, 6)
    q = o.rotate(np.repeat(x[1:2], 6, axis=0), np.arange(6) + 9, 100.0, 6)
    assert np.allclose((z * q).sum(-1), (z * q).sum(-1)[0])
    s = o.sink_softmax(np.array([[[0.0, -np.inf]]]), np.array([0.0]))
    assert np.allclose(s, [[[0.5, 0.0]]])
