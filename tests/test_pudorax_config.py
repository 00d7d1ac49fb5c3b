"""Pudorax without a GPU: configuration, spec and manifest, refusals, what the passes of a loop keep,
and the plain implementation's own properties."""
import copy
import math

import pytest
import torch

import plain_pudorax as plain
import pudorax_tiny as tiny
from cretif_b200.config import (ConfigError, build_pudorax_spec, pudorax_config_from_dict,
                                resolve_architecture)
from cretif_b200.engine.model import Model, manifest


def _spec(cfg):
    return build_pudorax_spec(pudorax_config_from_dict(cfg))


def test_registered_and_parsed():
    assert resolve_architecture("Pudorax").config_from_dict is pudorax_config_from_dict
    cfg = pudorax_config_from_dict(tiny.P_A)
    assert (cfg.vocab, cfg.width, cfg.eps, len(cfg.layers)) == (96, 64, 1e-5, 4)
    assert (cfg.embedding_scale, cfg.logit_softcap, cfg.token_side) == (3.0, 12.0, 8)
    assert cfg.loop == {"start": 1, "stop": 3, "times": 3}
    for raw in tiny.CONFIGS.values():
        c = pudorax_config_from_dict(raw)
        assert pudorax_config_from_dict(c.to_dict()).to_dict() == c.to_dict()


def test_parts_and_their_constants():
    spec = _spec(tiny.P_A)
    spec.validate()
    mixer, ff, side = spec.layers[0].branches
    assert mixer.norm.kind == ff.norm.kind == spec.final_norm.kind == "layernorm"
    assert side.norm is None and side.post_norm.kind == "rmsnorm" and mixer.post_norm is None
    p = mixer.part.params
    assert mixer.part.kind == "attention" and p["window"] == 0
    assert (p["num_heads"], p["num_kv_heads"], p["head_dim"], p["value_dim"], p["scale"]) == \
        (4, 2, 16, 24, 0.3)
    assert p["conv"]["taps"] == 3 and p["qk_norm"]["eps"] == 1e-5 and p["out_gate"] == "mix.g"
    assert p["position"] == {"kind": "rotary", "theta": 500.0, "rotary_dim": 8,
                             "pairing": "interleaved"}
    assert "position" not in _spec(tiny.P_D).layers[2].branches[0].part.params
    m = spec.layers[1].branches[0].part
    assert m.kind == "state_space" and (m.params["num_heads"], m.params["value_dim"],
                                        m.params["state_dim"], m.params["groups"],
                                        m.params["norm_groups"], m.params["conv_taps"]) == \
        (6, 16, 20, 3, 4, 4)
    r = ff.part.params
    assert (r["num_experts"], r["top"], r["intermediate_size"], r["scores"]) == \
        (7, 2, 32, "softmax_chosen")
    assert r["clamp"] == {"limit": 0.8, "slope": 1.702, "offset": 1.0}
    assert r["shared"]["clamp"] == {"limit": 1.3, "slope": 1.702, "offset": 1.0}
    assert r["router_bias"] == "mlp.router.b" and r["weight_on"] == "output"
    assert side.part.kind == "token_side" and side.part.params["dim"] == 8
    assert [l.branches[-1].part.params["part"] for l in spec.layers] == [0, 1, 2, 3]
    assert len(spec.layers[2].branches) == 2
    assert spec.embedding.params["scale"] == 3.0 and spec.head.params["softcap"] == 12.0
    assert spec.merge.kind == "linear_merge"
    bare = _spec(tiny.P_D)
    assert bare.merge is None and "softcap" not in bare.head.params
    assert all(b.part.kind != "token_side" for l in bare.layers for b in l.branches)
    assert "shared" not in bare.layers[1].branches[1].part.params


@pytest.mark.parametrize("name, order, merges", [
    ("A", [0, 1, 2, 1, 2, 1, 2, 3], [1, 3, 5]), ("B", [0, 1, 0, 1, 2, 3], [0, 2]),
    ("C", [0, 1, 2, 3], [2]), ("D", [0, 1, 2, 3], []), ("E", [0, 1, 2, 0, 1, 2], [0, 3])])
def test_the_order_of_layers_and_where_the_input_comes_in(name, order, merges):
    spec = _spec(tiny.CONFIGS[name])
    assert [e.layer for e in spec.schedule] == order
    assert [i for i, e in enumerate(spec.schedule) if e.merge_input] == merges
    assert all(e.cache is None and not e.add_input for e in spec.schedule)
    assert [(i, m) for i, m in plain.run_order(tiny.CONFIGS[name])] == \
        [(e.layer, e.merge_input) for e in spec.schedule]


def test_manifest_names_and_shapes():
    names, ignorable = manifest(_spec(tiny.P_A))
    shapes = {k: v.shape for k, v in names.items()}
    for name, shape in {
            "embed": (96, 64), "head": (96, 64), "side.embed": (96, 32), "loop.in": (64, 128),
            "final.norm": (64,), "final.norm.b": (64,), "l0.norm1": (64,), "l0.norm2.b": (64,),
            "l0.mix.q": (64, 64), "l0.mix.k": (32, 64), "l0.mix.v": (48, 64), "l0.mix.g": (96, 64),
            "l0.mix.o": (64, 96), "l0.mix.q.norm": (64,), "l0.mix.k.norm": (32,),
            "l0.mix.q.conv": (64, 3), "l0.mix.v.conv": (48, 3), "l1.mix.in": (318, 64),
            "l1.mix.conv": (216, 4), "l1.mix.conv.b": (216,), "l1.mix.dt_bias": (6,),
            "l1.mix.A_log": (6,), "l1.mix.D": (6,), "l1.mix.norm": (96,), "l1.mix.o": (64, 96),
            "l0.mlp.router": (7, 64), "l0.mlp.router.b": (7,), "l0.mlp.e6.gate": (32, 64),
            "l0.mlp.e0.down": (64, 32), "l0.mlp.shared.up": (48, 64), "l3.side.gate": (8, 64),
            "l3.side.proj": (64, 8), "l3.side.norm": (64,)}.items():
        assert shapes[name] == shape, name
    assert not ignorable
    for absent in ("l2.norm2", "l2.mlp.router", "l0.mlp.e7.gate", "l1.mix.q", "l0.side.embed"):
        assert absent not in shapes, absent
    bare = manifest(_spec(tiny.P_D))[0]
    assert "side.embed" not in bare and "loop.in" not in bare and "l0.side.norm" not in bare


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0].update(type="retention"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"].update(scale=0), "scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][1]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "top"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0), "limit"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(limit=-1.0), "limit"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["token_side"].update(dim=0), "dim"),
    (lambda c: c.update(logit_softcap=0.0), "logit_softcap"),
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_refusals(edit, text):
    cfg = copy.deepcopy(tiny.P_A)
    edit(cfg)
    with pytest.raises(ConfigError, match=text):
        pudorax_config_from_dict(cfg)


def test_every_pass_keeps_its_own():
    model = Model(_spec(tiny.P_A), torch.float32, "cpu")       # built, not loaded
    reqs = model.cache_requests()
    assert set(reqs) == {(i, 0) for i in range(8)}              # a mixer per schedule entry
    kv, inputs = reqs[(0, 0)]
    assert (kv.num_kv_heads, kv.head_dim, kv.value_dim, kv.window) == (2, 16, 24, 0)
    assert inputs.shape == ((64 + 32 + 48) * 2,)
    state = reqs[(1, 0)]
    assert state == reqs[(3, 0)] == reqs[(5, 0)]
    assert state.shape == (6 * 20 * 16 + 216 * 3,) and state.dtype == torch.float32
    assert model.graph_safe
    from cretif_b200.cache import SequenceCache
    cache = SequenceCache(reqs, 256, torch.float32, "cpu")
    views = [cache.state_view((i, 0)) for i in (1, 3, 5)]
    assert len({v.data_ptr() for v in views}) == 3
    assert len({cache.kv_view((i, 0)).k.data_ptr() for i in (2, 4, 6)}) == 3
    # one tap: nothing to keep beside the keys
    one = Model(_spec(tiny.P_C), torch.float32, "cpu").cache_requests()
    assert not isinstance(one[(0, 0)], tuple) and one[(1, 0)].shape == (4,)


def test_unknown_combinations_are_refused():
    from cretif_b200.config import PartSpec
    from cretif_b200.parts import build_part

    def build(category, kind, params):
        return build_part(category, PartSpec(kind, params), 16, torch.float32, "cpu")
    att = {"num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "scale": 1.0,
           "names": {"q": "q", "k": "k", "v": "v", "o": "o"}}
    conv = {"taps": 3, "q": "a", "k": "b", "v": "c"}
    norm = {"eps": 1e-5, "q": "d", "k": "e"}
    build("mixer", "attention", {**att, "conv": conv, "qk_norm": norm, "out_gate": "g"})
    for extra in ({"conv": conv}, {"conv": conv, "qk_norm": norm, "own_kv": False},
                  {"conv": conv, "qk_norm": norm, "chunk": 8},
                  {"conv": conv, "qk_norm": norm, "window": 8, "pool": 4},
                  {"conv": conv, "qk_norm": norm, "bias": {"q": "x", "k": "y", "v": "z"}},
                  {"conv": conv, "qk_norm": norm, "head_norm": {"eps": 1e-5}},
                  {"conv": conv, "head_norm": {"eps": 1e-5}, "out_gate": "g"},
                  {"out_gate": "g", "head_gate": "h"},
                  {"conv": {**conv, "taps": 0}, "qk_norm": norm}):
        with pytest.raises(ValueError):
            build("mixer", "attention", {**att, **extra})
    ssm = {"num_heads": 4, "groups": 2, "state_dim": 8, "value_dim": 6, "conv_taps": 4, "norm_groups": 3,
           "eps": 1e-5}
    build("mixer", "state_space", ssm)
    for extra in ({"groups": 3}, {"norm_groups": 5}, {"state_dim": 0}, {"state_dim": 1025},
                  {"conv_taps": 0}):
        with pytest.raises(ValueError):
            build("mixer", "state_space", {**ssm, **extra})
    moe = {"num_experts": 4, "top": 2, "intermediate_size": 8,
           "names": {"router": "r", "gate": "g{e}", "up": "u{e}", "down": "d{e}"}}
    for extra in ({"clamp": {"limit": 0.0}}, {"clamp": {"limit": 1.0}, "gated": False},
                  {"scores": "softmax_chosen", "correction": "c"},
                  {"scores": "softmax_chosen", "groups": {"count": 2, "keep": 1}}):
        with pytest.raises(ValueError):
            build("feed_forward", "routed_experts", {**moe, **extra})
    side = {"dim": 4, "part": 1, "parts": 2, "vocab_size": 9, "names": {}}
    for extra in ({"part": 2}, {"dim": 0}, {"activation": "step"}):
        with pytest.raises(ValueError):
            build("feed_forward", "token_side", {**side, **extra})
    spec = _spec(tiny.P_A)
    spec.merge = None
    with pytest.raises(ValueError, match="merge"):
        spec.validate()


def test_layers_share_the_second_embedding_and_keep_their_own_columns():
    from cretif_b200.weights.loader import random_weights
    spec = _spec(tiny.P_A)
    names, _ = manifest(spec)
    tensors = random_weights(names, 5, torch.bfloat16)
    model = Model(spec, torch.float32, "cpu")
    model.load(tensors)
    for i, layer in enumerate(model.layers):
        assert torch.equal(layer.branches[-1].part.table,
                           tensors["side.embed"].float()[:, 8 * i:8 * i + 8])


# ------------------------------------------------------------------ the plain implementation
def test_convolution_and_rotation():
    u = torch.tensor([[1.0], [2.0], [4.0], [8.0]], dtype=torch.float64)
    w = torch.tensor([[0.5, -1.0, 3.0]], dtype=torch.float64)
    # tap order: two before, one before, present
    assert plain.causal_conv(u, w).flatten().tolist() == [3.0, 5.0, 10.5, 21.0]
    z = torch.zeros(3, 1, 6, dtype=torch.float64)
    z[:, 0, 2] = 1.0
    r = plain.rotate_pairs(z, 100.0, 4)
    a = 2 * 100.0 ** -0.5
    assert torch.allclose(r[2, 0], torch.tensor([0, 0, math.cos(a), math.sin(a), 0, 0],
                                                dtype=torch.float64))
    assert torch.equal(plain.rotate_pairs(z, 100.0, 2), z)


def test_the_recurrence_is_a_decayed_sum():
    g = torch.Generator().manual_seed(0)
    S, H, G, N, e = 9, 4, 2, 5, 3
    x = torch.randn(S, H, e, generator=g, dtype=torch.float64)
    B, C = (torch.randn(S, G, N, generator=g, dtype=torch.float64) for _ in range(2))
    dt = torch.rand(S, H, generator=g, dtype=torch.float64)
    a, D = torch.rand(H, generator=g, dtype=torch.float64), torch.randn(H, generator=g, dtype=torch.float64)
    y = plain.state_space(x, B, C, dt, a, D)
    for h in range(H):
        for t in range(S):
            want = D[h] * x[t, h]
            for s in range(t + 1):
                want = want + math.exp(-float(a[h] * dt[s + 1:t + 1, h].sum())) * dt[s, h] \
                    * (C[t, h // 2] @ B[s, h // 2]) * x[s, h]
            assert torch.allclose(y[t, h], want)


def test_norms_gates_and_choices():
    x = torch.tensor([[1.0, 2.0, 3.0, 6.0]], dtype=torch.float64)
    n = plain.centred(x, 1e-9)
    assert abs(float(n.mean())) < 1e-12 and abs(float((n * n).mean()) - 1) < 1e-6
    y = plain.gated_parts_norm(x, torch.full_like(x, 50.0), 2, torch.ones(4, dtype=torch.float64), 0.0)
    assert torch.allclose((y.reshape(2, 2) ** 2).mean(dim=-1), torch.ones(2, dtype=torch.float64))
    ids, w = plain.choose(torch.tensor([0.0, 2.0, -1.0, 2.0 + math.log(3.0)], dtype=torch.float64), 2)
    assert ids == [3, 1] and torch.allclose(w, torch.tensor([0.75, 0.25], dtype=torch.float64))
    eye = torch.eye(2, dtype=torch.float64)
    W = {"gate": eye, "up": eye * -1, "down": eye}
    got = plain.clamped_expert(torch.tensor([5.0, -5.0], dtype=torch.float64), W, "", 2.0)
    # the gate is clamped from above only, the other product on both sides
    want = [2.0 / (1 + math.exp(-3.404)) * -1.0, -5.0 / (1 + math.exp(8.51)) * 3.0]
    assert torch.allclose(got, torch.tensor(want, dtype=torch.float64))


def test_a_pass_more_is_another_model():
    from cretif_b200.weights.loader import random_weights
    cfg = copy.deepcopy(tiny.P_A)
    names, _ = manifest(_spec(cfg))
    w = {k: v.double() for k, v in random_weights(names, 3, torch.bfloat16).items()}
    streams = []
    one = plain.forward(cfg, w, [3, 1, 4, 1, 5], streams=streams)
    assert len(streams) == 8
    cfg["loop"]["times"] = 2
    assert (plain.forward(cfg, w, [3, 1, 4, 1, 5]) - one).abs().max() > 1e-6


def test_the_bench_configurations_build():
    import importlib.util
    import os
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bench.py")
    mod_spec = importlib.util.spec_from_file_location("bench_for_pudorax", path)
    bench = importlib.util.module_from_spec(mod_spec)
    mod_spec.loader.exec_module(bench)
    for z in bench.DESIGN_SIZES.values():
        configs = bench.pudorax_configs(z, 4)
        assert {"losorax attention routed", "virorax retention", "gibipel routed"} < set(configs)
        ssm = configs["pudorax mamba2"]["layers"][0]["mixer"]
        ret = configs["virorax retention"]["layers"][0]["mixer"]
        assert ssm["heads"] * ssm["vdim"] == ret["heads"] * ret["vdim"] and ssm["state"] == ret["dim"]
        for name, cfg in configs.items():
            if name.startswith("pudorax"):
                spec = _spec(cfg)
                spec.validate()
                assert len(spec.schedule) == (6 if "looped" in name else 4)
