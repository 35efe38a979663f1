"""Small seeded Mubopel models for the tests: (shape, weights as float64, checkpoint folder)."""
import os

from tests.conftest import CACHE, synth_module
from tests.latent_oracle import widen


def shapes():
    s = synth_module()
    L = s.LatentLayer
    return {
        # two kinds of layers, one of them without a feed-forward, borrowed rows
        "mixed": s.LatentShape(96, 210, [L(scale=0.3), L(kv_from=0, heads=3, dim=24, vdim=40, q_rank=20, ff=0, scale=0.3),
                                         L(heads=2, dim=16, rot_dim=8, vdim=48, q_rank=64, kv_rank=24, ff=72, base=500.0, scale=0.5),
                                         L(kv_from=2, heads=5, dim=8, rot_dim=8, vdim=8, q_rank=16, kv_rank=24, ff=96, base=500.0, scale=0.5)],
                               eps=1e-3, residual_mult=0.7),
        # nothing a multiple of 8, a borrower behind two lenders
        "odd": s.LatentShape(100, 203, [L(heads=3, dim=20, rot_dim=6, vdim=12, q_rank=23, kv_rank=37, ff=53, scale=0.4),
                                        L(heads=1, dim=9, rot_dim=10, vdim=21, q_rank=10, kv_rank=18, ff=30, base=77.0, scale=0.4),
                                        L(kv_from=0, heads=7, dim=5, rot_dim=6, vdim=3, q_rank=8, kv_rank=37, ff=11, scale=0.4)], residual_mult=1.0),
        # head sizes and ranks of a large model (several row tiles of the decode attention, two blocks of 64 columns per operand)
        "big": s.LatentShape(256, 520, [L(heads=20, dim=128, rot_dim=64, vdim=128, q_rank=192, kv_rank=512, ff=640, scale=0.2),
                                        L(heads=20, dim=80, rot_dim=32, vdim=160, q_rank=100, kv_rank=256, ff=320, scale=0.3)], residual_mult=0.4),
        # beyond what the split attention holds: one (token, head) per CTA, prompts through the narrow path
        "huge": s.LatentShape(64, 96, [L(heads=2, dim=48, rot_dim=16, vdim=272, q_rank=32, kv_rank=640, ff=64, scale=0.4)]),
        # vocabulary beyond one pass of the head's CTAs, many layers of different rotations
        "wide_vocab": s.LatentShape(64, 9000, [L(heads=2, dim=16, rot_dim=8, vdim=16, q_rank=16, kv_rank=32, ff=32, base=10.0 ** (1 + i), scale=0.3) for i in range(10)]),
    }


def model(name, seed=5):
    s = synth_module()
    shape = shapes()[name]
    bits = s.random_weights(shape, seed)
    path = os.path.join(CACHE, f"latent_{name}_{seed}_{os.getpid()}")
    if not os.path.exists(os.path.join(path, "config.json")):
        s.write_checkpoint(path, shape, weights=bits)
    return shape, {k: widen(v) for k, v in bits.items()}, path
