"""Small seeded Baporax models for the tests: (shape, weights as float64, checkpoint folder)."""
import os

from tests.conftest import CACHE, synth_module
from tests.hybrid_oracle import widen


def shapes():
    s = synth_module()
    S, A, H = s.SsmLayer, s.DiffLayer, s.HybridShape
    return {
        # a loop in the middle, a window of a few tokens and one wider than a key tile
        "looped": H(96, 210, [S(), A(window=9), S(heads=6, vdim=16, state=48, groups=3, norm_groups=1, ff=0), A(heads=3, kv_heads=1, window=77, dim=16, vdim=48, diff=0.2)],
                    loop=(1, 3, 3), eps=1e-3, logit_scale=0.3),
        # nothing a multiple of 8, parts of the gated norm that cut through heads, one tap, no loop, other filter lengths
        "odd": H(100, 203, [A(heads=5, kv_heads=5, dim=9, vdim=13, window=33, conv=1, diff=0.7, ff=51), S(heads=3, vdim=10, state=7, groups=1, norm_groups=5, conv=2, ff=37),
                            S(heads=5, vdim=7, state=70, groups=5, norm_groups=1, conv=5, ff=0), A(heads=2, kv_heads=1, dim=70, vdim=20, window=1, conv=7, ff=29)]),
        # head sizes of a large model; everything looped, from the first layer on
        "big": H(256, 520, [S(heads=10, vdim=64, state=128, groups=2, norm_groups=2, ff=512), A(heads=8, kv_heads=2, dim=64, vdim=128, window=200, ff=384)], loop=(0, 2, 2), logit_scale=4.0),
        # beyond what the prompt kernels hold: wide values, states of 200 columns with wide heads
        "huge": H(64, 96, [A(heads=2, kv_heads=1, dim=144, vdim=272, window=40, ff=64), S(heads=2, vdim=144, state=250, groups=1, norm_groups=2, ff=64)], loop=(1, 2, 1)),
        # many layers of few, large CTAs: kernels of several layers are resident at once, and finished scores wait for slow products
        "deep": H(128, 120, [A(heads=16, kv_heads=4, dim=64, vdim=128, window=150, ff=512) for _ in range(8)] + [S(heads=24, vdim=64, state=128, groups=4, norm_groups=4, ff=512)]),
        # one kind of layer each, no feed-forward anywhere; a vocabulary beyond one pass of the head's CTAs
        "states": H(64, 9000, [S(heads=8, vdim=16, state=16, groups=8, norm_groups=8, ff=0) for _ in range(2)], loop=(0, 1, 4), logit_scale=1.7),
        "windows": H(72, 150, [A(heads=6, kv_heads=2, dim=24, vdim=24, window=64 + i, ff=0) for i in range(3)], loop=(2, 3, 2)),
    }


def model(name, seed=5):
    s = synth_module()
    shape = shapes()[name]
    bits = s.random_weights(shape, seed)
    path = os.path.join(CACHE, f"hybrid_{name}_{seed}_{os.getpid()}")
    if not os.path.exists(os.path.join(path, "config.json")):
        s.write_checkpoint(path, shape, weights=bits)
    return shape, {k: widen(v) for k, v in bits.items()}, path
