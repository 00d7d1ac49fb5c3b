"""Tiny Gibipel configurations for the tests; they differ in every size, order and option."""
import numpy as np


def _left(heads, kv, dim, vdim, window, pool, scale, rot_dims, base=10000.0, scaling=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
         "mask": {"size": window, "pool": pool}, "rot": {"base": base, "dims": rot_dims}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def _right(heads, dim, vdim, cap=9.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def _mixer(left, right, a=1.0, b=1.0):
    return {"left": left, "right": right, "left_scale": a, "right_scale": b}


def _moe(experts, top, ff, identity=None, groups=None, shared=None):
    router = {"experts": experts, "top": top}
    if identity is not None:
        router["identity"] = identity
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _model(vocab, width, eps, layers, embed=1.0, logit=1.0, positions=1024):
    return {"architecture": "Gibipel", "vocab": vocab, "width": width, "max_positions": positions,
            "norm": {"eps": eps}, "embedding": {"scale": embed}, "logit_scale": logit,
            "layers": [{"type": "parallel", "mixer": m, "mlp": f} for m, f in layers]}


# small windows and blocks of sizes that divide nothing, values wider and narrower than keys, a part
# of each head rotated, experts with identities in groups, a layer without a feed-forward
G_A = _model(96, 64, 1e-5, [
    (_mixer(_left(4, 2, 16, 24, 9, 4, 0.4, 8, 500.0, (4.0, 1.0, 4.0, 60)), _right(4, 16, 24), 1.2, 0.7),
     _moe(10, 3, 32, identity=2, groups=(4, 3), shared=48)),
    (_mixer(_left(4, 1, 16, 8, 21, 5, 0.3, 16), _right(2, 32, 16, 6.0), 0.5, 1.4), None),
    (_mixer(_left(2, 2, 24, 24, 13, 13, 0.35, 12, 300.0, (8.0, 2.0, 3.0, 100)), _right(3, 8, 32), 0.9, 1.1),
     _moe(7, 2, 40, identity=3)),
], embed=3.0, logit=0.7)
# sizes the tensor-core kernels take in bfloat16 (heads of 64 and 128), windows and blocks that cross
# cache blocks, blocks longer than the window, one expert a token, no identities
G_B = _model(130, 96, 1e-6, [
    (_mixer(_left(4, 2, 64, 64, 70, 16, 0.15, 64, 5000.0, (4.0, 1.0, 4.0, 300)), _right(2, 64, 64), 0.8, 1.3),
     _moe(8, 1, 64, groups=(2, 1), shared=64)),
    (_mixer(_left(2, 1, 128, 128, 20, 48, 0.1, 64), _right(3, 32, 48, 20.0), 1.3, 0.6),
     _moe(6, 2, 64, identity=2)),
    (_mixer(_left(6, 2, 32, 32, 130, 3, 0.2, 16), _right(1, 128, 80), 1.0, 1.0), None),
], embed=2.0, logit=1.5)
# everything that can be one is one: one head, a window that shows a query nothing but itself, blocks
# of one token, one expert, groups of one, a rotation of one pair, factors of one
G_C = _model(70, 48, 1e-5, [
    (_mixer(_left(1, 1, 8, 8, 1, 1, 1.0, 2), _right(1, 8, 8, 1.0)), _moe(1, 1, 16)),
    (_mixer(_left(1, 1, 16, 8, 2, 1, 0.5, 16), _right(1, 4, 16, 3.0)),
     _moe(3, 2, 24, identity=1, groups=(4, 3), shared=8)),
    (_mixer(_left(1, 1, 8, 16, 1, 6, 0.7, 8), _right(1, 16, 1)), _moe(1, 1, 8, identity=1)),
])
# sizes that are multiples of nothing in particular, a window longer than any test sequence, a factor
# below zero, a mixer that is left out by its factor, every group kept, more identities than experts
G_D = _model(77, 36, 1e-5, [
    (_mixer(_left(3, 1, 12, 20, 500, 7, 0.29, 4), _right(3, 6, 10), -0.6, 1.2),
     _moe(2, 3, 20, identity=4, groups=(2, 2))),
    (_mixer(_left(2, 2, 20, 6, 33, 10, 0.3, 10), _right(5, 12, 7, 30.0), 1.1, 0.0), None),
    (_mixer(_left(5, 5, 4, 4, 3, 2, 0.8, 4), _right(1, 20, 12), 0.0, 1.7),
     _moe(5, 2, 28, shared=12)),
], embed=0.5, logit=-2.0)
# windows and blocks of a cache block and one more or less; more than eight query heads on a
# key/value head
G_E = _model(200, 128, 1e-6, [
    (_mixer(_left(16, 1, 64, 64, 64, 64, 0.12, 32), _right(2, 64, 128), 0.7, 0.9),
     _moe(12, 4, 64, identity=4, groups=(4, 2), shared=128)),
    (_mixer(_left(4, 4, 64, 64, 65, 8, 0.11, 64), _right(4, 16, 16), 1.0, 0.8), None),
    (_mixer(_left(12, 1, 32, 32, 63, 1, 0.2, 32), _right(2, 20, 32), 1.1, 1.2),
     _moe(30, 6, 48, identity=2)),
], embed=4.0, logit=0.5)

CONFIGS = {"A": G_A, "B": G_B, "C": G_C, "D": G_D, "E": G_E}
SEEDS = {"A": 61, "B": 62, "C": 63, "D": 64, "E": 65}


def one_layer(side, mixer=None, mlp=None, vocab=64, width=64):
    """A model of one layer in which only one of the two mixers counts ("left" or "right"; the
    other's factor is zero), or both ("both")."""
    if mixer is None:
        mixer = _mixer(_left(4, 2, 16, 16, 12, 4, 0.4, 8), _right(4, 16, 16),
                       0.0 if side == "right" else 1.0, 0.0 if side == "left" else 1.0)
    return _model(vocab, width, 1e-5, [(mixer, mlp)], positions=4096)


def tokens(name, n, seed):
    rng = np.random.default_rng(7000 * seed + n)
    return rng.integers(0, CONFIGS[name]["vocab"], size=n).tolist()
