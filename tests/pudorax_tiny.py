"""Tiny Pudorax configurations for the tests; they differ in every size, order and option."""
import numpy as np


def _att(heads, kv, dim, vdim, scale, conv, rot_dims, base=10000.0):
    return "attention", {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
                         "conv": conv, "rot": {"base": base, "dims": rot_dims}}


def _ssm(heads, vdim, state, groups=1, norm_groups=1, conv=4):
    return "mamba2", {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                      "norm_groups": norm_groups, "conv": conv}


def _moe(experts, top, ff, limit, shared=None, shared_limit=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit},
         "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def _model(vocab, width, eps, layers, scale=1.0, loop=None, side=None, cap=None, positions=1024):
    cfg = {"architecture": "Pudorax", "vocab": vocab, "width": width, "max_positions": positions,
           "norm": {"eps": eps}, "embedding": {"scale": scale},
           "layers": [{"type": m[0], "mixer": m[1], "mlp": f} for m, f in layers]}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    if side is not None:
        cfg["token_side"] = {"dim": side}
    if cap is not None:
        cfg["logit_softcap"] = cap
    return cfg


# values wider and narrower than keys, taps of every number, groups and parts that do not coincide, a
# layer without a feed-forward, a loop in the middle
P_A = _model(96, 64, 1e-5, [
    (_att(4, 2, 16, 24, 0.3, 3, 8, 500.0), _moe(7, 2, 32, 0.8, 48, 1.3)),
    (_ssm(6, 16, 20, 3, 4, 4), _moe(5, 3, 24, 1.1, 16, 0.6)),
    (_att(4, 1, 16, 8, 0.4, 2, 16), None),
    (_ssm(2, 32, 16, 1, 2, 2), _moe(4, 1, 40, 0.9, 32, 2.0)),
], scale=3.0, loop=(1, 3, 3), side=8, cap=12.0)
# sizes the tensor-core kernels take in bfloat16 (heads of 64 and 128), states for the chunks of 64
# tokens, the loop from the first layer on, one expert a token
P_B = _model(130, 96, 1e-6, [
    (_ssm(4, 64, 64, 2, 1, 4), _moe(8, 1, 64, 1.5, 64, 1.0)),
    (_att(4, 2, 64, 64, 0.12, 4, 64, 5000.0), _moe(6, 2, 64, 1.2, 64, 0.7)),
    (_att(2, 1, 128, 128, 0.09, 3, 32), _moe(4, 4, 128, 2.0)),
    (_ssm(2, 48, 32, 2, 2, 3), None),
], scale=2.0, loop=(0, 2, 2), side=64, cap=20.0)
# everything that can be one is one: heads, groups, taps, experts, a pass, state channels
P_C = _model(70, 48, 1e-5, [
    (_att(1, 1, 8, 8, 1.0, 1, 2), _moe(1, 1, 16, 1.0, 8, 1.0)),
    (_ssm(1, 1, 1, 1, 1, 1), _moe(3, 3, 8, 0.5)),
    (_ssm(1, 16, 4, 1, 1, 2), None),
    (_att(1, 1, 8, 16, 0.5, 2, 8), _moe(1, 1, 8, 3.0)),
], loop=(2, 3, 1), side=1, cap=5.0)
# sizes that are multiples of nothing in particular, no loop, no side, no cap, nothing rotated, more
# taps than tokens in many portions
P_D = _model(77, 36, 1e-5, [
    (_att(3, 1, 12, 20, 0.29, 6, 4), _moe(5, 2, 20, 0.7, 12, 0.4)),
    (_ssm(3, 10, 6, 3, 3, 7), _moe(2, 2, 28, 1.0)),
    (_att(5, 5, 4, 6, 0.8, 5, 0), None),
    (_ssm(5, 7, 12, 1, 5, 5), _moe(9, 4, 10, 1.7, 14, 0.9)),
], scale=0.5)
# more than eight query heads on a key/value head, the loop over every layer, a state wider than a head
P_E = _model(200, 128, 1e-6, [
    (_ssm(8, 16, 128, 4, 8, 4), _moe(12, 4, 64, 1.0, 128, 1.5)),
    (_att(16, 1, 64, 64, 0.12, 4, 32), _moe(30, 6, 48, 0.6, 48, 0.8)),
    (_ssm(4, 64, 32, 1, 1, 3), _moe(6, 2, 64, 2.5, 64, 2.5)),
], scale=4.0, loop=(0, 3, 2), side=24, cap=30.0)

CONFIGS = {"A": P_A, "B": P_B, "C": P_C, "D": P_D, "E": P_E}
SEEDS = {"A": 71, "B": 72, "C": 73, "D": 74, "E": 75}


def one_layer(mixer, mlp=None, vocab=64, width=64, **options):
    return _model(vocab, width, 1e-5, [(mixer, mlp)], positions=4096, **options)


def tokens(name, n, seed):
    rng = np.random.default_rng(9000 * seed + n)
    return rng.integers(0, CONFIGS[name]["vocab"], size=n).tolist()
