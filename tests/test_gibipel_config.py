"""Gibipel without a GPU: configuration, spec and manifest, refusals, the cache's pooled entries, and
the plain implementation's own properties."""
import copy
import math

import pytest
import torch

import gibipel_tiny as tiny
import plain_gibipel as plain
from cretif_b200.config import (ConfigError, build_gibipel_spec, gibipel_config_from_dict,
                                resolve_architecture)
from cretif_b200.engine.model import Model, manifest


def _spec(cfg):
    return build_gibipel_spec(gibipel_config_from_dict(cfg))


def test_registered_and_parsed():
    assert resolve_architecture("Gibipel").config_from_dict is gibipel_config_from_dict
    cfg = gibipel_config_from_dict(tiny.G_A)
    assert (cfg.vocab, cfg.width, cfg.eps, len(cfg.layers)) == (96, 64, 1e-5, 3)
    assert (cfg.embedding_scale, cfg.logit_scale) == (3.0, 0.7)
    assert gibipel_config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()


def test_parts_and_their_constants():
    spec = _spec(tiny.G_A)
    spec.validate()
    for layer in spec.layers:
        for b in layer.branches:
            assert b.norm is None and b.post_norm.kind == "rmsnorm" and b.post_norm.params["scalar"]
    mixer, ff = (b.part for b in spec.layers[0].branches)
    assert mixer.kind == "parallel" and ff.kind == "routed_experts"
    left, right = mixer.params["sides"]
    assert (left["name"], left["kind"], left["scale"]) == ("left", "attention", 1.2)
    assert (right["name"], right["kind"], right["scale"]) == ("right", "matrix_memory", 0.7)
    p = left["params"]
    assert (p["window"], p["pool"], p["head_dim"], p["value_dim"], p["scale"]) == (9, 4, 16, 24, 0.4)
    assert p["position"] == {"kind": "rotary", "theta": 500.0, "rotary_dim": 8, "pairing": "half",
                             "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 60.0}}
    assert "scaling" not in _spec(tiny.G_A).layers[1].branches[0].part.params["sides"][0]["params"]["position"]
    assert right["params"]["gate_cap"] == 9.0
    r = ff.params
    assert (r["num_experts"], r["identities"], r["top"], r["scores"]) == (10, 2, 3, "softmax")
    assert r["groups"] == {"count": 4, "keep": 3, "score": "best"} and r["renormalize"]
    assert r["correction"] == "mlp.correction" and r["sum_eps"] == 1e-20
    assert r["weight_on"] == "output" and r["shared"]["intermediate_size"] == 48
    assert len(spec.layers[1].branches) == 1
    last = spec.layers[2].branches[1].part.params
    assert "groups" not in last and "shared" not in last and last["identities"] == 3
    assert spec.embedding.params["scale"] == 3.0 and spec.head.params["scale"] == 0.7
    assert not spec.head.params["tied"] and spec.final_norm.params["scalar"]


def test_manifest_names_and_shapes():
    names, ignorable = manifest(_spec(tiny.G_A))
    shapes = {k: v.shape for k, v in names.items()}
    for name, shape in {
            "embed": (96, 64), "head": (96, 64), "final.norm": (), "l0.norm1": (), "l0.norm2": (),
            "l0.mix.left.q": (64, 64), "l0.mix.left.q.b": (64,), "l0.mix.left.q.norm": (64,),
            "l0.mix.left.k": (32, 64), "l0.mix.left.k.norm": (32,), "l0.mix.left.v": (48, 64),
            "l0.mix.left.v.b": (48,), "l0.mix.left.sink": (4,), "l0.mix.left.o": (64, 96),
            "l0.mix.right.q": (64, 64), "l0.mix.right.v": (96, 64), "l0.mix.right.g": (96, 64),
            "l0.mix.right.i": (4, 64), "l0.mix.right.i.b": (4,), "l0.mix.right.f.b": (4,),
            "l0.mix.right.norm": (96,), "l0.mix.right.o": (64, 96),
            "l0.mlp.router": (12, 64), "l0.mlp.correction": (12,), "l0.mlp.e9.gate": (32, 64),
            "l0.mlp.e0.down": (64, 32), "l0.mlp.shared.up": (48, 64),
            "l2.mlp.router": (10, 64)}.items():
        assert shapes[name] == shape, name
    assert not ignorable
    for absent in ("l1.norm2", "l1.mlp.router", "l0.mlp.e10.gate", "l2.mlp.shared.gate"):
        assert absent not in shapes, absent


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].pop("pool"), "pool"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=3), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("factor"), "factor"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(low=4.0), "low"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=0), "gate_cap"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=13), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=3), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=5), "groups"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c.pop("logit_scale"), "logit_scale"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
])
def test_refusals(edit, text):
    cfg = copy.deepcopy(tiny.G_A)
    edit(cfg)
    with pytest.raises(ConfigError, match=text):
        gibipel_config_from_dict(cfg)


def test_each_side_keeps_what_it_asks_for():
    model = Model(_spec(tiny.G_A), torch.float32, "cpu")       # built, not loaded
    reqs = model.cache_requests()
    assert set(reqs) == {(i, 0, s) for i in range(3) for s in ("left", "right")}
    kv, state = reqs[(0, 0, "left")], reqs[(0, 0, "right")]
    assert (kv.num_kv_heads, kv.head_dim, kv.value_dim, kv.window, kv.pool) == (2, 16, 24, 9, 4)
    assert state.shape[0] >= 4 * (16 * 24 + 16 + 1) and state.shape[0] % 4 == 0
    assert model.graph_safe


def test_unknown_combinations_are_refused():
    from cretif_b200.parts import build_part
    from cretif_b200.config import PartSpec
    base = {"num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "scale": 1.0,
            "names": {"q": "q", "k": "k", "v": "v", "o": "o"}}
    for extra in ({"pool": 4}, {"pool": 4, "chunk": 8}, {"pool": 4, "window": 8, "own_kv": False},
                  {"out_scale": 2.0}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("attention", {**base, **extra}), 16, torch.float32, "cpu")
    moe = {"num_experts": 4, "top": 2, "intermediate_size": 8,
           "names": {"router": "r", "gate": "g{e}", "up": "u{e}", "down": "d{e}"}}
    for extra in ({"scores": "linear"}, {"identities": 2, "weight_on": "input"},
                  {"identities": 1, "groups": {"count": 2, "keep": 1}},
                  {"groups": {"count": 2, "keep": 1, "score": "median"}}):
        with pytest.raises(ValueError):
            build_part("feed_forward", PartSpec("routed_experts", {**moe, **extra}), 16,
                       torch.float32, "cpu")


# ------------------------------------------------------------------ the cache's pooled entries
def test_blocks_for_entries_and_a_window_that_waits_for_its_block():
    from cretif_b200.cache import KVRequest, SequenceCache
    # a window of 20 tokens, an entry for every 48: the tokens of an unfinished block must stay
    cache = SequenceCache({(0, 0, "a"): KVRequest(2, 16, 20, pool=48)}, max_tokens=64 * 200,
                          dtype=torch.float32, device="cpu", block_tokens=16, max_slots=4)
    view = cache.kv_view((0, 0, "a"))
    assert view.pool.pool == 48 and view.pool.k.shape[1:] == view.k.shape[1:] == (2, 16, 16)
    s = cache.alloc_slot()
    tokens, entries = cache._kv_groups
    length = 0
    for n in (47, 1, 1, 95, 1, 623, 1, 1):
        cache.begin_step([(s, n)])
        # every entry of a block that is complete after the step has a place
        done = (length + n) // 48
        assert all(entries.table_host[s, e // 16] >= 0 for e in range(done)), length
        # and the tokens of the block that this step may complete are all still there
        first = length // 48 * 48
        assert all(tokens.table_host[s, p // 16] >= 0 for p in range(first, length + n)), length
        assert all(tokens.table_host[s, p // 16] >= 0
                   for p in range(max(0, length - 20 + 1), length + n))
        cache.end_step([(s, n)])
        length += n
        cache.check()
    assert int(tokens.first_block[s]) > 0                        # old tokens were given back
    assert entries.pool.held_count == -(-(length // 48) // 16)
    cache.free_slot(s)
    assert all(g.pool.held_count == 0 for g in cache._kv_groups)
    cache.check()


def test_entries_never_run_out_before_tokens_do():
    """Whatever lengths the live sequences have, the tokens' own limit is reached first."""
    from cretif_b200.cache import CacheFull, KVRequest, SequenceCache
    for pool in (1, 3, 16, 64, 100):
        for lens in ([16] * 40, [17] * 40, [640], [639, 1], [300, 300], [pool] * 40, [33] * 9):
            cache = SequenceCache({0: KVRequest(1, 16, 1 << 20, pool=pool)}, max_tokens=640,
                                  dtype=torch.float32, device="cpu", block_tokens=16)
            held = 0
            for n in lens:
                need = -(-n // 16)
                if held + need > 40:
                    break
                s = cache.alloc_slot()
                cache.begin_step([(s, n)])                       # must not raise
                cache.end_step([(s, n)])
                held += need
            cache.check()
    cache = SequenceCache({0: KVRequest(1, 16, 8, pool=4)}, max_tokens=64, dtype=torch.float32,
                          device="cpu", block_tokens=16)
    s = cache.alloc_slot()
    with pytest.raises(CacheFull):
        cache.begin_step([(s, 65)])
    cache.reserve(s, 64)                                         # entries are mapped ahead
    assert cache._kv_groups[1].pool.held_count == 1


def test_stretched_wavelengths_in_the_rotation_table():
    from cretif_b200.parts.position import rotary_table, stretched_frequencies
    for base, dims, sc in ((10000.0, 64, (4.0, 1.0, 4.0, 300)), (500.0, 10, (8.0, 2.0, 3.0, 100)),
                           (3.0, 2, (2.0, 0.5, 50.0, 7))):
        scaling = dict(zip(("factor", "low", "high", "original"), sc))
        f = plain.frequencies(base, dims, scaling)
        cos, sin = rotary_table(base, dims, 50, "cpu", scaling)
        ang = torch.arange(50, dtype=torch.float64)[:, None] * f[None, :]
        assert (cos.double() - torch.cos(ang)).abs().max() < 1e-6
        assert (sin.double() - torch.sin(ang)).abs().max() < 1e-6
        assert not torch.allclose(cos, rotary_table(base, dims, 50, "cpu")[0])
    with pytest.raises(ValueError):
        stretched_frequencies(f, {"factor": 2.0, "low": 3.0, "high": 3.0, "original": 8})


# ------------------------------------------------------------------ the plain implementation
def test_what_a_window_with_blocks_shows():
    tok, blk = plain.window_and_blocks(20, 5, 3)
    assert tok[10].nonzero().flatten().tolist() == [6, 7, 8, 9, 10]
    # tokens 0 .. 5 lie before the window: blocks 0 and 1 (0..2, 3..5)
    assert blk[10].nonzero().flatten().tolist() == [0, 1]
    assert blk[9].nonzero().flatten().tolist() == [0]             # 3, 4 have left, 5 has not
    assert blk[7].nonzero().flatten().tolist() == [0] and not blk[6].any()
    tok, blk = plain.window_and_blocks(6, 1, 1)
    assert tok.sum() == 6 and blk[3].nonzero().flatten().tolist() == [0, 1, 2]
    rows = torch.arange(7.0)[:, None]
    assert plain.block_means(rows, 3).flatten().tolist() == [1.0, 4.0]


def test_wavelengths():
    f = plain.frequencies(100.0, 8)
    assert torch.allclose(f, torch.tensor([1.0, 100.0 ** -0.25, 0.1, 100.0 ** -0.75],
                                          dtype=torch.float64))
    sc = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 40.0}
    g = plain.frequencies(100.0, 8, sc)
    # wavelengths 6.3, 19.9, 62.8, 198.7: kept below 10, stretched above 40, blended between
    assert float(g[0]) == 1.0
    assert torch.allclose(g[2:], f[2:] / 4.0)
    s = (40.0 / (2 * math.pi / float(f[1])) - 1.0) / 3.0
    assert abs(float(g[1]) - ((1 - s) * float(f[1]) / 4.0 + s * float(f[1]))) < 1e-12


def test_the_running_maximum_changes_nothing_but_the_floor():
    """Against the recurrence without it: S = sum of prod(exp f) exp(i) k v^T, and the floor of the
    denominator is exp(-m) in stabilised units, which is one in plain ones as long as m is the
    reference of all of them."""
    g = torch.Generator().manual_seed(0)
    S, d, e = 25, 5, 4
    q, k, v = (torch.randn(S, 1, n, generator=g, dtype=torch.float64) for n in (d, d, e))
    i = torch.randn(S, 1, generator=g, dtype=torch.float64) * 3
    f = plain.log_sigmoid(torch.randn(S, 1, generator=g, dtype=torch.float64) * 2)
    got = plain.memory(q, k, v, i, f)[:, 0]
    M, n, m = torch.zeros(d, e, dtype=torch.float64), torch.zeros(d, dtype=torch.float64), 0.0
    for t in range(S):
        M = math.exp(f[t]) * M + math.exp(i[t]) * torch.outer(k[t, 0], v[t, 0])
        n = math.exp(f[t]) * n + math.exp(i[t]) * k[t, 0]
        m = max(float(f[t]) + m, float(i[t]))
        den = max(abs(float(n @ q[t, 0])), 1.0) + 1e-6 * math.exp(m)
        assert torch.allclose(got[t], M.T @ q[t, 0] / den)


def test_choices():
    s = torch.tensor([0.3, 0.1, 0.05, 0.25, 0.2, 0.1], dtype=torch.float64)
    zero = torch.zeros(6, dtype=torch.float64)
    assert plain.choose(s, zero, 2) == [0, 3]
    c = torch.tensor([-0.5, 0.0, 0.0, 0.0, 0.0, 0.3], dtype=torch.float64)
    assert plain.choose(s, c, 2) == [5, 3]                        # the correction decides
    # groups of two, scored by their best: 0.3, 0.25, 0.2
    assert plain.choose(s, zero, 3, {"count": 3, "keep": 2}) == [0, 3, 1]
    # all choice scores below zero: what is left out stays out
    assert plain.choose(s, zero - 2.0, 2, {"count": 3, "keep": 1}) == [0, 1]


def test_identities_and_weights():
    g = torch.Generator().manual_seed(1)
    mlp = {"router": {"experts": 2, "top": 2, "identity": 2}}
    W = {"p.router": torch.zeros(4, 6, dtype=torch.float64),
         "p.correction": torch.tensor([0.0, -9.0, 5.0, -9.0], dtype=torch.float64)}
    for e in range(2):
        for n, sh in (("gate", (3, 6)), ("up", (3, 6)), ("down", (6, 3))):
            W[f"p.e{e}.{n}"] = torch.randn(sh, generator=g, dtype=torch.float64)
    h = torch.randn(2, 6, generator=g, dtype=torch.float64)
    y = plain.routed(h, W, "p.", mlp)                             # equal scores: identity 2, expert 0
    for t in range(2):
        assert torch.allclose(y[t], 0.5 * h[t] + 0.5 * plain.gated(h[t], W, "p.e0."))


def test_the_bench_configurations_build():
    import importlib.util
    import os
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bench.py")
    mod_spec = importlib.util.spec_from_file_location("bench_for_gibipel", path)
    bench = importlib.util.module_from_spec(mod_spec)
    mod_spec.loader.exec_module(bench)
    for z in bench.DESIGN_SIZES.values():
        configs = bench.gibipel_configs(z, 4)
        assert {"virorax attention", "virorax retention", "losorax attention routed"} < set(configs)
        for name, cfg in configs.items():
            if name.startswith("gibipel"):
                spec = _spec(cfg)
                spec.validate()
                assert len(spec.schedule) == 4 and spec.architecture == "Gibipel"
                left = cfg["layers"][0]["mixer"]["left"]
                other = configs["virorax attention"]["layers"][0]["mixer"]
                assert all(left[k] == other[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale"))
                assert left["mask"]["size"] == other["mask"]["size"]
