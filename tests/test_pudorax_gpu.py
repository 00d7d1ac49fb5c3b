"""Pudorax through the engine against the plain implementation (``plain_pudorax``): every mechanism
alone, every way of cutting requests into steps, far keys and far memory, the first tokens of a
sequence, reused slots, greedy generation through the library's own entry point."""
import json
import os

import numpy as np
import pytest
import torch

import plain_pudorax as plain
import pudorax_tiny as tiny
from replay_cuts import (rel_err, run_batch, run_chunks, run_schedule, run_tail_by_one,
                         run_whole)

pytestmark = pytest.mark.gpu

# Relative to the largest plain logit.  The float32 runs are the sharp ones.  bfloat16 rounds
# activations, keys and values to eight bits several times a layer: its bound is on the median over
# the positions, with a loose one on nine in ten.  In a model with routed experts a choice that is a
# close call may fall the other way under that rounding, which changes the position's output by an
# expert and shows at later positions through keys and states: twice the bounds.
TOL = {"float32": 1e-4, "bfloat16": 4e-2}
BF16_MOST = 0.25
I32 = dict(dtype=torch.int32, device="cuda")


def close(got, want, dtype, slack=1.0):
    if dtype == "float32":
        return rel_err(got, want) <= TOL[dtype]
    want = np.asarray(want, dtype=np.float64)
    per_row = np.abs(np.asarray(got, dtype=np.float64) - want).max(axis=-1) / np.abs(want).max()
    ok = (np.median(per_row) <= slack * TOL[dtype]
          and np.quantile(per_row, 0.9) <= slack * BF16_MOST)
    if not ok:
        print("per row:", np.round(np.sort(per_row)[::-1][:8], 3), "median", np.median(per_row))
    return ok


def close_routed(got, want, dtype):
    return close(got, want, dtype, slack=2.0)


LENGTHS = {"A": [1, 2, 3, 10, 23, 75, 140], "B": [2, 5, 64, 65, 131, 200], "C": [1, 2, 9, 40],
           "D": [1, 4, 31, 70, 100], "E": [1, 2, 33, 129, 200]}
WIDE = (".q", ".k", ".v", ".g", ".o", ".in", ".up", ".gate", ".down", ".proj", ".router")


def _write(tmp_path_factory, name, cfg, seed, edit=None):
    """A model folder for ``cfg`` with seeded random weights; ``edit(tensors)`` may change
    tensors before they are written."""
    from cretif_b200.config import build_pudorax_spec, pudorax_config_from_dict
    from cretif_b200.engine.model import manifest
    from cretif_b200.weights.loader import random_weights, write_model_folder
    d = str(tmp_path_factory.mktemp(f"pudorax_{name}"))
    names, _ = manifest(build_pudorax_spec(pudorax_config_from_dict(cfg)))
    tensors = random_weights(names, seed, torch.bfloat16)
    # wider projections than the default draw: scores, gates and clamps that are not all alike
    for k in tensors:
        if k in ("embed", "head"):
            tensors[k] = (tensors[k].float() * 20.0).to(torch.bfloat16)
        elif k.endswith(WIDE) and k != "loop.in" and "router" not in k:
            tensors[k] = (tensors[k].float() * 6.0).to(torch.bfloat16)
        elif k.endswith(".b"):
            tensors[k] = (tensors[k].float() * 10.0 if "norm" in k else tensors[k].float()
                          ).to(torch.bfloat16)
    if edit is not None:
        edit(tensors)
    write_model_folder(d, cfg, tensors)
    return d


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {n: _write(tmp_path_factory, n, c, tiny.SEEDS[n]) for n, c in tiny.CONFIGS.items()}


@pytest.fixture(scope="module")
def engines(folders):
    from cretif_b200.engine import Engine
    made = {}

    def get(name, dtype, max_tokens=2048):
        key = (name, dtype, max_tokens)
        if key not in made:
            made[key] = Engine(folders[name], dtype=dtype, max_tokens=max_tokens)
        return made[key]
    return get


@pytest.fixture(scope="module")
def plain_logits(folders):
    models, memo = {}, {}

    def get(name, toks):
        key = (name, tuple(toks))
        if key not in memo:
            if name not in models:
                models[name] = plain.read_model_folder(folders[name])
            cfg, w = models[name]
            memo[key] = plain.forward(cfg, w, list(toks)).numpy()
        return memo[key]
    return get


# ------------------------------------------------------------------ registry and loading
def test_the_configuration_picks_the_model_and_its_parts(folders):
    from cretif_b200.config import load_config
    from cretif_b200.engine import Engine
    arch, cfg, spec = load_config(folders["A"])
    assert arch.name == "Pudorax" and spec.vocab_size == 96 and spec.hidden_size == 64
    eng = Engine(folders["A"], dtype="float32", max_tokens=256)
    groups = eng.cache.stats()["groups"]
    # one attention layer that runs once, one that runs in three passes
    assert sorted((g["head_dim"], g["value_dim"], g["window"], g["layers"]) for g in groups) == \
        [(16, 8, 0, 3), (16, 24, 0, 1)]
    assert eng.cache.stats()["state_bytes"] > 0


# ------------------------------------------------------------------ kernels of the mechanisms
@pytest.mark.parametrize("R,H", [(1, 2048), (5, 516), (255, 3000), (256, 1024), (300, 2052), (3, 4096),
                                 (2, 514), (700, 35), (1, 8), (400, 96)])
def test_layer_norm(R, H):
    """Few and many rows, with and without a branch to add first, gathered rows, both element types;
    rows whose mean is large beside their spread."""
    from cretif_b200.csrc import ops
    g = torch.Generator().manual_seed(R + H)
    h = torch.randn(R, H, generator=g) + 30.0 * torch.randn(R, 1, generator=g)
    w, b = torch.randn(H, generator=g), torch.randn(H, generator=g)
    for dt in (torch.float32, torch.bfloat16):
        for ddt in (None, torch.float32, torch.bfloat16):
            delta = None if ddt is None else (torch.randn(R, H, generator=g) * 2).to(ddt)
            v = h.double() + (0 if delta is None else delta.double())
            want = plain.centred(v, 1e-5) * w.double() + b.double()
            hc = h.cuda()
            out = torch.empty(R, H, dtype=dt, device="cuda")
            ops.add_layernorm(hc, None if delta is None else delta.cuda(), w.cuda(), b.cuda(), out, 1e-5)
            tol = 2e-4 if dt == torch.float32 else 4e-2
            assert (out.cpu().double() - want).abs().max() < tol, (dt, ddt)
            assert (hc.cpu().double() - v).abs().max() < 1e-5
        rows = torch.randint(0, R, (9,), generator=g, dtype=torch.int32)
        out = torch.empty(9, H, dtype=dt, device="cuda")
        ops.add_layernorm(h.cuda(), None, w.cuda(), b.cuda(), out, 1e-5, rows=rows.cuda())
        want = plain.centred(h[rows.long()].double(), 1e-5) * w.double() + b.double()
        assert (out.cpu().double() - want).abs().max() < (2e-4 if dt == torch.float32 else 4e-2)


@pytest.mark.parametrize("stream", [False, True])
@pytest.mark.parametrize("M,K,N", [(1, 64, 40), (3, 576, 100), (9, 2048, 130), (20, 512, 64), (33, 96, 50),
                                   (64, 1032, 24), (64, 256, 17), (2, 8, 8), (8, 4104, 16)])
def test_layer_norm_in_the_few_token_products(M, K, N, stream):
    """The prologue against the norm's own kernel (the same rounding to bfloat16) and the plain norm;
    weights through registers and through shared memory, rows shared by a cluster or not, gathered."""
    from cretif_b200.csrc import ops
    g = torch.Generator().manual_seed(M * K)
    h = torch.randn(M + 3, K, generator=g) + 3.0 * torch.randn(M + 3, 1, generator=g)
    nw, nb = torch.randn(K, generator=g) * 0.3 + 1, torch.randn(K, generator=g)
    w = (torch.randn(N, K, generator=g) * K ** -0.5).bfloat16()
    if not ops.fused_supported(M, K, w.cuda(), norm=2):
        pytest.skip("the rows do not fit the kernel's shared memory")
    old_k, old_b = ops.set_stream_min_k(1 if stream else 1 << 30), ops.stream_min_bytes()
    ops.set_stream_min_k(1 if stream else 1 << 30, 1 << 60)
    try:
        for rows in (None, torch.randint(0, M + 3, (M,), generator=g, dtype=torch.int32)):
            src = h[:M] if rows is None else h[rows.long()]
            x = (plain.centred(src.double(), 1e-5) * nw.double() + nb.double()).bfloat16().double()
            want = x @ w.double().T
            hc = h[:M].contiguous().cuda() if rows is None else h.cuda()
            for dt in (torch.float32, torch.bfloat16):
                out = torch.empty(M, N, dtype=dt, device="cuda")
                ops.fused_norm_linear(hc, nw.cuda(), 1e-5, w.cuda(), out,
                                      rows=None if rows is None else rows.cuda(), norm_b=nb.cuda())
                # (a value on the border of two bfloat16 numbers may fall either way)
                assert (out.cpu().double() - want).abs().max() <= 1e-2 * want.abs().max(), (dt, stream)
            act = torch.empty(M, N, dtype=torch.float32, device="cuda")
            ops.fused_norm_linear(hc, nw.cuda(), 1e-5, w.cuda(), act, unary="gelu_tanh", alpha=0.5,
                                  rows=None if rows is None else rows.cuda(), norm_b=nb.cuda())
            ref = plain.gelu_tanh(0.5 * want)
            assert (act.cpu().double() - ref).abs().max() <= 1e-2 * max(1.0, float(ref.abs().max()))
    finally:
        ops.set_stream_min_k(old_k, old_b)


def test_a_layer_norm_in_front_of_the_head():
    from cretif_b200.config import PartSpec
    from cretif_b200.parts import build_part
    g = torch.Generator().manual_seed(2)
    H, V = 64, 48
    w = (torch.randn(V, H, generator=g) * 0.4).bfloat16()
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        head = build_part("head", PartSpec("linear_head", {"tied": False, "name": "head", "softcap": 2.0,
                                                           "vocab_size": V}), H, dtype, "cuda")
        head.load({"weight": w})
        norm = build_part("norm", PartSpec("layernorm", {"eps": 1e-6, "name": "n"}), H, dtype, "cuda")
        norm.load({"weight": torch.rand(H, generator=g) + 0.5, "bias": torch.randn(H, generator=g)})
        for R in (1, 7, 200):
            h = torch.randn(R, H, generator=g) + 1.0
            z = (plain.centred(h.double(), 1e-6) * norm.weight.cpu().double()
                 + norm.bias.cpu().double()) @ w.double().T
            want = 2.0 * torch.tanh(z / 2.0)
            got = head.forward_from_residual(h.cuda(), None, norm, None, None)
            assert (got is not None) == (dtype == torch.bfloat16 and R <= 64)
            if got is not None:
                assert (got.cpu().double() - want).abs().max() <= tol * want.abs().max()
            got = head.forward(norm.forward(h.cuda(), None), None)
            assert (got.cpu().double() - want).abs().max() <= tol * want.abs().max(), (dtype, R)


def _table(positions, bt=64):
    n = (positions + bt - 1) // bt + 1
    return n, (torch.arange(1, n + 1, dtype=torch.int32, device="cuda").flip(0)[None, :] - 1
               ).contiguous()


def _cache_for(positions, nkv, hd, dtype, bt=64):
    n, table = _table(positions, bt)
    return torch.zeros(n, nkv, bt, hd, dtype=dtype, device="cuda"), table


def _gather(cache, table, positions, bt=64):
    t = table[0].cpu()
    return torch.stack([cache[t[p // bt], :, p % bt].cpu() for p in range(positions)])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,e,rot,pairing,taps", [
    (4, 2, 16, 24, 8, 1, 3), (2, 1, 64, 64, 64, 1, 4), (3, 1, 12, 20, 4, 1, 2), (5, 5, 20, 6, 10, 1, 3),
    (1, 1, 8, 8, 2, 1, 1), (8, 2, 128, 128, 32, 1, 4), (2, 2, 16, 16, 0, 1, 6), (4, 1, 32, 32, 16, 0, 3),
    (1, 1, 9, 5, 2, 1, 5)])
def test_convolution_norms_over_whole_projections_rotation_and_cache_write(dtype, H, G, d, e, rot, pairing,
                                                                           taps):
    """The kernel between an attention's input product and its scores over a sequence fed in pieces of
    every kind (shorter than the convolution's reach, single tokens in a row, long ones), and the saved
    inputs that it and the prompt's kernel leave."""
    from cretif_b200.csrc import ops
    from cretif_b200.parts.position import rotary_table
    g = torch.Generator().manual_seed(4)
    S, base, eps = 300, 300.0, 1e-5
    C = (H + G) * d + G * e
    proj = torch.randn(S, C + 3, generator=g) * 2
    conv = torch.randn(C, taps, generator=g)
    wq, wk = torch.randn(H * d, generator=g), torch.randn(G * d, generator=g)
    rows = plain.causal_conv(proj[:, :C].double(), conv.double())
    q = (plain.unit(rows[:, :H * d], eps) * wq.double()).reshape(S, H, d)
    k = (plain.unit(rows[:, H * d:(H + G) * d], eps) * wk.double()).reshape(S, G, d)
    v = rows[:, (H + G) * d:].reshape(S, G, e)
    cos = sin = None
    if rot:
        cos, sin = rotary_table(base, rot, S, torch.device("cuda"))
        perm = list(range(d))
        if pairing == 0:             # pair (i, i + rot/2): the same rotation after a permutation
            perm = [x for i in range(rot // 2) for x in (i, i + rot // 2)] + list(range(rot, d))
        inv = np.argsort(perm)
        q = plain.rotate_pairs(q[..., perm], base, rot)[..., inv]
        k = plain.rotate_pairs(k[..., perm], base, rot)[..., inv]
    kc, table = _cache_for(S, G, d, dtype)
    vc, _ = _cache_for(S, G, e, dtype)
    keep = taps - 1
    width = -(-C * keep // 4) * 4
    state = torch.zeros(3, max(4, width), device="cuda")
    state[1:] = 7.0                                     # other slots' inputs
    fault = torch.zeros(1, dtype=torch.int32, device="cuda")
    q_out = torch.zeros(S, H * d, dtype=dtype, device="cuda")
    at = 0
    for n in (1, 2, 30, 1, 1, 1, 1, 200, 2, 1, 3) + (1,) * 57:
        pos, zeros = torch.arange(at, at + n, **I32), torch.zeros(n, **I32)
        start = torch.tensor([at], **I32)
        p = proj[at:at + n].cuda()
        ops.projnorm_rope_kv_append(
            p, None, wq.cuda(), wk.cuda(), eps, cos, sin, pairing, rot, pos, zeros, zeros[:1], H, G, d, e,
            q_out[at:at + n], table=table, kc=kc, vc=vc, fault=fault,
            conv=(conv.t().contiguous().cuda(), state if keep else None, start, n == 1))
        if n > 1 and keep:
            ops.delta_conv_state(p, state, taps, C, torch.tensor([0, n], **I32), zeros[:1], 1)
        at += n
        for j in range(keep):                           # oldest first, zeros before the start
            back = at - keep + j
            want = proj[back, :C] if back >= 0 else torch.zeros(C)
            assert torch.equal(state[0, :C * keep].cpu().reshape(C, keep)[:, j], want), (at, j)
    assert at == S and int(fault.item()) == 0
    assert bool((state[1:] == 7.0).all())
    tol = 2e-4 if dtype == torch.float32 else 8e-2
    assert (q_out.cpu().double().reshape(S, H, d) - q).abs().max() < tol
    ks, vs = _gather(kc, table, S).double(), _gather(vc, table, S).double()
    assert (ks - k).abs().max() < tol and (vs - v).abs().max() < tol * max(1.0, float(v.abs().max()) / 8)


def _ssm_case(seed, S, H, G, N, e, taps, wild):
    """Projected rows and weights; ``wild``: step sizes from almost none to ones that wipe the state,
    decays from none to sudden."""
    g = torch.Generator().manual_seed(seed)
    inner, C = H * e, H * e + 2 * G * N
    rows = torch.randn(S, inner + C + H, generator=g)
    if wild:
        rows[:, -H:] = rows[:, -H:] * 6 - 2
        rows[S // 3::S // 3 + 1, -H:] = 30.0
    p = dict(conv=torch.randn(C, taps, generator=g) * 0.6, conv_b=torch.randn(C, generator=g) * 0.3,
             a_log=torch.randn(H, generator=g) * (2.0 if wild else 0.7),
             dt_bias=torch.randn(H, generator=g) - 1, D=torch.randn(H, generator=g),
             norm=torch.randn(inner, generator=g))
    return rows, p


def _ssm_want(rows, p, H, G, N, e, parts, eps):
    inner, C = H * e, H * e + 2 * G * N
    d = {k: v.double() for k, v in p.items()}
    u = rows.double()
    S = u.shape[0]
    xbc = plain.silu(plain.causal_conv(u[:, inner:inner + C], d["conv"]) + d["conv_b"])
    y = plain.state_space(xbc[:, :inner].reshape(S, H, e), xbc[:, inner:inner + G * N].reshape(S, G, N),
                          xbc[:, inner + G * N:].reshape(S, G, N),
                          plain.softplus(u[:, inner + C:] + d["dt_bias"]), torch.exp(d["a_log"]), d["D"])
    return plain.gated_parts_norm(y.reshape(S, inner), u[:, :inner], parts, d["norm"], eps)


class _Ssm:
    """The kernels over slots of a state, in pieces."""

    def __init__(self, p, H, G, N, e, parts, taps, slots=3, eps=1e-5):
        self.p, self.sizes, self.parts, self.taps, self.eps = p, (H, G, N, e), parts, taps, eps
        self.C = H * e + 2 * G * N
        self.at = -(-H * N * e // 4) * 4
        self.state = torch.zeros(slots, self.at + -(-self.C * (taps - 1) // 4) * 4, device="cuda")
        self.c = {k: v.contiguous().cuda() for k, v in p.items() if k != "conv"}
        self.w = p["conv"].t().contiguous().cuda()

    def run(self, rows, slot, cu, form="auto", dtype=torch.float32, write=True):
        from cretif_b200.csrc import ops
        H, G, N, e = self.sizes
        B, T = len(cu) - 1, rows.shape[0]
        out = torch.empty(T, H * e, dtype=dtype, device="cuda")
        seq = torch.repeat_interleave(torch.arange(B), torch.tensor(cu).diff()).to(torch.int32).cuda()
        cu_d, slot_d = torch.tensor(cu, **I32), torch.tensor(slot, **I32)
        r = rows.cuda()
        save = T == B and self.taps > 1 and write
        ops.state_space(r, self.w, self.c["conv_b"], self.c["a_log"], self.c["dt_bias"], self.c["D"],
                        self.state, self.at, cu_d, slot_d, seq, B, H, G, N, e, self.parts,
                        self.c["norm"], self.eps, out, write_state=write, save_inputs=save, form=form)
        if self.taps > 1 and write and not save:
            ops.delta_conv_state(r[:, H * e:], self.state[:, self.at:], self.taps, self.C, cu_d, slot_d, B)
        return out.cpu()


@pytest.mark.parametrize("wild", [False, True])
@pytest.mark.parametrize("H,G,N,e,parts,taps", [
    (4, 2, 64, 64, 2, 4), (6, 3, 20, 16, 4, 3), (2, 1, 128, 32, 1, 2), (3, 3, 32, 48, 3, 4),
    (8, 1, 16, 16, 8, 1), (5, 5, 12, 7, 1, 5), (1, 1, 256, 80, 5, 4), (16, 2, 32, 64, 1, 4)])
def test_state_space_in_both_forms(H, G, N, e, parts, taps, wild):
    """Chunks of 64 tokens and token by token against the recurrence written out, over a sequence fed in
    pieces that end inside chunks; the same state from both, other slots untouched."""
    S = 211
    rows, p = _ssm_case(H * N, S, H, G, N, e, taps, wild)
    want = _ssm_want(rows, p, H, G, N, e, parts, 1e-5)
    chunkable = N % 4 == 0 and e % 16 == 0
    states = []
    for form in ("token", "chunk", "auto") if chunkable else ("token", "auto"):
        for cuts in ([S], [1, 2, 3, 61, 65, 1, 1, 77]):
            k = _Ssm(p, H, G, N, e, parts, taps)
            k.state[0] = k.state[2] = 5.0
            at, got = 0, []
            for n in cuts:
                got.append(k.run(rows[at:at + n], [1], [0, n], form))
                at += n
            got = torch.cat(got).double()
            assert (got - want).abs().max() <= 2e-4 * want.abs().max(), (form, cuts, wild)
            assert bool((k.state[0] == 5.0).all() and (k.state[2] == 5.0).all())
            states.append(k.state[1, :H * N * e].cpu())
            keep = taps - 1
            saved = k.state[1, k.at:k.at + k.C * keep].cpu().reshape(k.C, keep)
            assert torch.equal(saved, rows[S - keep:, H * e:H * e + k.C].t())
    for s in states[1:]:
        assert (s - states[0]).abs().max() <= 1e-4 * states[0].abs().max()
    k = _Ssm(p, H, G, N, e, parts, taps)
    half = k.run(rows, [1], [0, S], dtype=torch.bfloat16).double()
    assert (half - want).abs().max() <= 1e-2 * want.abs().max()


def test_state_space_of_unequal_sequences_in_one_step():
    """Several sequences with portions of every length in the steps, slots in any order; each as alone."""
    H, G, N, e, parts, taps = 4, 2, 32, 32, 2, 4
    lens = [1, 64, 3, 130, 65, 2, 17]
    rows, p = _ssm_case(5, sum(lens) + 40, H, G, N, e, taps, True)
    seqs, at = [], 0
    for n in lens:
        seqs.append(rows[at:at + n + 3])
        at += n
    slots = [4, 0, 6, 2, 9, 1, 7]
    for form in ("auto", "token", "chunk"):
        k = _Ssm(p, H, G, N, e, parts, taps, slots=10)
        cu = [0] + list(np.cumsum(lens))
        got = k.run(torch.cat([s[:n] for s, n in zip(seqs, lens)]), slots, cu, form)
        parts_ = [[got[cu[i]:cu[i + 1]]] for i in range(7)]
        for step in range(3):                         # and three single tokens each
            out = k.run(torch.stack([s[n + step] for s, n in zip(seqs, lens)]), slots, list(range(8)))
            for i in range(7):
                parts_[i].append(out[i:i + 1])
        for i, s in enumerate(seqs):
            want = _ssm_want(s, p, H, G, N, e, parts, 1e-5)
            err = (torch.cat(parts_[i]).double() - want).abs().max()
            assert err <= 3e-4 * want.abs().max(), (form, i, float(err))
        assert bool((k.state[[3, 5, 8]] == 0).all())


def test_state_space_leaves_the_state_alone_when_asked():
    H, G, N, e = 2, 1, 16, 16
    rows, p = _ssm_case(6, 90, H, G, N, e, 4, False)
    for form in ("token", "chunk"):
        k = _Ssm(p, H, G, N, e, 1, 4)
        k.state.normal_()
        before = k.state.clone()
        out = k.run(rows, [1], [0, 90], form, write=False)
        assert torch.equal(k.state, before) and bool(torch.isfinite(out).all())
        k.run(rows, [1], [0, 90], form)
        assert not torch.equal(k.state[1], before[1])


def test_state_space_refuses_what_it_does_not_take():
    from cretif_b200.csrc.ops import KernelError
    H, G, N, e = 2, 1, 6, 16
    rows, p = _ssm_case(7, 80, H, G, N, e, 4, False)
    k = _Ssm(p, H, G, N, e, 1, 4)
    with pytest.raises(KernelError):
        k.run(rows, [1], [0, 80], "chunk")             # a state that 16-byte accesses do not fit
    with pytest.raises(KernelError):
        k.run(rows[:, :-1], [1], [0, 80])
    k.parts = 3
    with pytest.raises(KernelError):
        k.run(rows, [1], [0, 80])


@pytest.mark.parametrize("E,top", [(20, 4), (8, 2), (3, 3), (1, 1), (64, 6), (256, 8), (40, 33)])
def test_routing_by_the_softmax_over_the_chosen(E, top):
    from cretif_b200.csrc import ops
    g = torch.Generator().manual_seed(E + top)
    T, H = 70, 48
    x, router = torch.randn(T, H, generator=g), torch.randn(E, H, generator=g) * 0.4
    # logits far below zero and far apart: a softmax over all would leave nothing of the last ones
    for bias in (torch.randn(E, generator=g), torch.randn(E, generator=g) * 60 - 200):
        z = x.double() @ router.double().T + bias.double()
        for way in ("route", "topk"):
            ids = torch.zeros(T, top, dtype=torch.int32, device="cuda")
            wts = torch.zeros(T, top, dtype=torch.float32, device="cuda")
            rule = dict(renorm=True, softmax="chosen", bias=bias.cuda())
            if way == "route":
                ops.moe_route(x.cuda(), router.cuda(), top, ids, wts, **rule)
            else:
                ops.moe_topk((x.double() @ router.double().T).float().cuda(), top, ids, wts, **rule)
            for t in range(T):
                want, w = plain.choose(z[t], top)
                got = dict(zip(ids[t].tolist(), wts[t].tolist()))
                assert set(got) == set(want), (way, t)
                assert all(abs(got[e] - float(b)) < 2e-5 for e, b in zip(want, w)), (way, t)


@pytest.mark.parametrize("limit", [0.6, 3.0])
@pytest.mark.parametrize("I,K", [(64, 64), (128, 96), (48, 40), (20, 33)])
def test_a_clamped_gate_in_every_product(I, K, limit):
    """A lone gated feed-forward with a clamped gate through the kernels for few and many rows, in both
    element types, beside the same part with SiLU."""
    from cretif_b200.config import PartSpec
    from cretif_b200.parts import build_part
    g = torch.Generator().manual_seed(I)
    w = {"gate": torch.randn(I, K, generator=g) * 0.3, "up": torch.randn(I, K, generator=g) * 0.3,
         "down": torch.randn(K, I, generator=g) * 0.3}
    w = {k: v.bfloat16() for k, v in w.items()}
    d = {k: v.double() for k, v in w.items()}
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 3e-2)):
        for clamp in ({"limit": limit, "slope": 1.702, "offset": 1.0},
                      {"limit": limit, "slope": 0.5, "offset": -0.3}, None):
            extra = {} if clamp is None else {"clamp": clamp}
            part = build_part("feed_forward", PartSpec("gated_mlp", {
                "intermediate_size": I, "names": {"gate": "g", "up": "u", "down": "d"}, **extra}), K,
                dtype, "cuda")
            part.load(w)
            for T in (1, 7, 50, 200):
                x = (torch.randn(T, K, generator=g) * 2).to(dtype)
                a, u = x.double() @ d["gate"].T, x.double() @ d["up"].T
                if clamp is None:
                    act = plain.silu(a) * u
                else:
                    a = a.clamp(max=limit)
                    act = a * plain.sigmoid(clamp["slope"] * a) * (u.clamp(-limit, limit)
                                                                   + clamp["offset"])
                want = act @ d["down"].T
                got = part.forward(x.cuda(), None)
                assert (got.cpu().double() - want).abs().max() <= tol * want.abs().max(), (dtype, T, clamp)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mlp", [tiny._moe(6, 2, 64, 0.8, 32, 1.5), tiny._moe(10, 3, 40, 1.2),
                                 tiny._moe(4, 4, 128, 0.5, 64, 0.5), tiny._moe(3, 1, 24, 2.0, 20, 0.7)])
def test_experts_through_every_product(tmp_path_factory, mlp, dtype):
    """A handful of pairs, sorted pairs and (in bfloat16) whole tiles on the tensor cores."""
    from cretif_b200.csrc import ops
    from cretif_b200.engine import Engine
    from cretif_b200.parts.experts import few_pairs_off

    def edit(tensors):
        # (logits far apart: no choice is a close call)
        tensors["l0.mlp.router"] = (tensors["l0.mlp.router"].float() * 2).to(torch.bfloat16)
    cfg = tiny.one_layer(tiny._att(4, 2, 16, 16, 0.3, 2, 8), mlp, side=8)
    d = _write(tmp_path_factory, "experts", cfg, seed=5, edit=edit)
    eng = Engine(d, dtype=dtype, max_tokens=1024, step_graphs=False)
    pcfg, w = plain.read_model_folder(d)
    toks = np.random.default_rng(6).integers(0, cfg["vocab"], size=150).tolist()
    want = plain.forward(pcfg, w, toks).numpy()
    # the clamps and the bias count: without them the logits are others
    loose = json.loads(json.dumps(pcfg))
    loose["layers"][0]["mlp"]["expert"]["limit"] = 1e9
    assert rel_err(plain.forward(loose, w, toks).numpy(), want) > 0.01
    if mlp["router"]["experts"] > mlp["router"]["top"]:
        other = {**w, "l0.mlp.router.b": -w["l0.mlp.router.b"]}
        assert rel_err(plain.forward(pcfg, other, toks).numpy(), want) > 0.01
    for few_off in (False, True):
        try:
            few_pairs_off(few_off)
            assert close_routed(run_whole(eng, toks), want, dtype), few_off
            assert close_routed(run_chunks(eng, toks, [3, 1, 1, 7, 60]), want, dtype), few_off
        finally:
            few_pairs_off(False)
    try:
        ops.moe_simt_only(True)
        assert close_routed(run_whole(eng, toks), want, dtype)
    finally:
        ops.moe_simt_only(False)


def test_the_combination_into_the_stream():
    """The experts' rows summed into the residual stream, which leaves its copy for the next reader."""
    from cretif_b200.csrc import ops
    g = torch.Generator().manual_seed(3)
    for T, H, top in ((1, 64, 2), (70, 36, 3), (5, 35, 1)):
        rows, y = torch.randn(T * top, H, generator=g), torch.randn(T, H, generator=g)
        wts, plus = torch.rand(T, top, generator=g), torch.randn(T, H, generator=g)
        yc, x = y.cuda(), torch.empty(T, H, dtype=torch.bfloat16, device="cuda")
        ops.moe_combine(rows.cuda(), None, top, yc, wts=wts.cuda(), plus=plus.cuda(), add=True, x_out=x)
        want = y.double() + plus.double() + (rows.double().reshape(T, top, H)
                                             * wts.double()[..., None]).sum(1)
        assert (yc.cpu().double() - want).abs().max() < 1e-5
        assert torch.equal(x, yc.to(torch.bfloat16))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim,width", [(8, 64), (64, 96), (24, 40), (1, 48), (13, 33)])
def test_a_second_look_at_the_token(dim, width, dtype):
    from cretif_b200.config import PartSpec
    from cretif_b200.parts import build_part

    class Ctx:
        pass
    g = torch.Generator().manual_seed(dim)
    V = 50
    part = build_part("feed_forward", PartSpec("token_side", {
        "dim": dim, "part": 1, "parts": 3, "vocab_size": V,
        "names": {"table": "/t", "gate": "g", "proj": "p"}}), width, dtype, "cuda")
    W = {"side.embed": torch.randn(V, 3 * dim, generator=g).bfloat16(),
         "p.side.gate": (torch.randn(dim, width, generator=g) * 0.4).bfloat16(),
         "p.side.proj": torch.randn(width, dim, generator=g).bfloat16(),
         "p.side.norm": torch.ones(width)}
    part.load({"table": W["side.embed"], "gate": W["p.side.gate"], "proj": W["p.side.proj"]})
    W = {k: v.double() for k, v in W.items()}
    for T in (1, 9, 64, 150):
        x = torch.randn(T, width, generator=g).to(dtype)
        ids = torch.randint(0, V, (T,), generator=g, dtype=torch.int32)
        ctx = Ctx()
        ctx.tok_ids = ids.cuda()
        y = part.forward(x.cuda(), ctx).cpu().double()
        got = plain.unit(y, 1e-6)
        want = plain.token_side(x.double(), ids.tolist(), W, "p.", 1, dim, 1e-6)
        # (a narrow gate may leave a row of next to nothing, which the norm blows up)
        e = torch.stack([W["side.embed"][t, dim:2 * dim] for t in ids.tolist()])
        raw = (plain.gelu_tanh(x.double() @ W["p.side.gate"].T) * e) @ W["p.side.proj"].T
        assert (y - raw).abs().max() <= (1e-5 if dtype == torch.float32 else 2e-2) * raw.abs().max()
        if dtype == torch.float32:
            loud = raw.abs().max(dim=1).values > 1e-2 * raw.abs().max()
            assert (got - want)[loud].abs().max() < 1e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [64, 96, 33])
def test_merging_the_input_in(width, dtype):
    from cretif_b200.config import PartSpec
    from cretif_b200.parts import build_part
    g = torch.Generator().manual_seed(width)
    part = build_part("merge", PartSpec("linear_merge", {"name": "w"}), width, dtype, "cuda")
    w = (torch.randn(width, 2 * width, generator=g) * 0.2).bfloat16()
    part.load({"weight": w})
    for T in (1, 9, 64, 150):
        x0 = torch.randn(T, width, generator=g)
        h = x0.cuda()
        rows = part.begin(h)
        want = x0.double()
        for _ in range(3):
            h += 1.0
            want = torch.cat([want + 1.0, x0.double()], dim=1) @ w.double().T
            part.forward(h, rows)
            assert (h.cpu().double() - want).abs().max() <= \
                (1e-5 if dtype == torch.float32 else 2e-2) * want.abs().max()


# ------------------------------------------------------------------ each mixer alone in a model
MIXERS = {"attention": tiny._att(4, 2, 16, 16, 0.4, 3, 8), "wide values": tiny._att(4, 1, 16, 24, 0.3, 4, 16),
          "heads of 64": tiny._att(4, 2, 64, 64, 0.15, 2, 32), "one tap": tiny._att(2, 2, 32, 32, 0.2, 1, 4),
          "mamba2": tiny._ssm(4, 16, 16, 2, 2), "state of 20": tiny._ssm(2, 24, 20, 1, 1, 3),
          "one tap of it": tiny._ssm(4, 16, 32, 4, 1, 1)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(MIXERS))
def test_one_layer_of_each_mixer(tmp_path_factory, which, dtype):
    from cretif_b200.engine import Engine
    cfg = tiny.one_layer(MIXERS[which])
    d = _write(tmp_path_factory, "one", cfg, seed=9)
    eng = Engine(d, dtype=dtype, max_tokens=1024)
    pcfg, w = plain.read_model_folder(d)
    rng = np.random.default_rng(3)
    for n in (1, 2, 13, 90):
        toks = rng.integers(0, cfg["vocab"], size=n).tolist()
        want = plain.forward(pcfg, w, toks).numpy()
        assert close(run_whole(eng, toks), want, dtype), (which, n)
        assert close(run_tail_by_one(eng, toks, tail=n), want, dtype), (which, n)
        assert close(run_chunks(eng, toks, [2, 5, 2, 30]), want, dtype), (which, n)
    eng.cache.check()


def test_mixers_of_this_design_stand_beside_one_another():
    """Both offer what lies between their products, so the side-by-side mixer takes them too."""
    from cretif_b200.config import PartSpec
    from cretif_b200.parts import build_part
    from cretif_b200.config import build_pudorax_spec, pudorax_config_from_dict
    sides = []
    for name, m in (("a", tiny._att(2, 1, 16, 16, 0.3, 3, 8)), ("b", tiny._ssm(2, 16, 16))):
        spec = build_pudorax_spec(pudorax_config_from_dict(tiny.one_layer(m)))
        part = spec.layers[0].branches[0].part
        sides.append({"name": name, "kind": part.kind, "params": part.params, "scale": 1.0})
    both = build_part("mixer", PartSpec("parallel", {"sides": sides}), 64, torch.float32, "cuda")
    assert both.together


@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_the_stream_after_every_layer(engines, folders, name):
    eng = engines(name, "float32")
    pcfg, w = plain.read_model_folder(folders[name])
    toks = tiny.tokens(name, 60, 7)
    want = []
    plain.forward(pcfg, w, toks, streams=want)
    got = []
    slot = eng.alloc_slot()
    eng.step([(slot, toks)], "all", streams=got)
    eng.free_slot(slot)
    assert len(got) == len(want)
    for i, (a, b) in enumerate(zip(got, want)):
        assert (a.cpu().double() - b).abs().max() <= 1e-4 * float(b.abs().max()), (name, i)


# ------------------------------------------------------------------ ways of cutting the work
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_whole_and_token_by_token(engines, plain_logits, name, dtype):
    eng = engines(name, dtype)
    for n in LENGTHS[name]:
        toks = tiny.tokens(name, n, 1)
        want = plain_logits(name, toks)
        got = run_whole(eng, toks)
        assert got.shape == want.shape
        assert close_routed(got, want, dtype), (name, n)
        assert close_routed(run_tail_by_one(eng, toks, tail=32), want, dtype), (name, n)
    toks = tiny.tokens(name, 20, 2)                    # nothing but single tokens
    assert close_routed(run_tail_by_one(eng, toks, tail=20), plain_logits(name, toks), dtype)
    eng.cache.check()


@pytest.mark.parametrize("name", ["A", "B", "E"])
def test_few_token_steps_with_and_without_the_fused_kernels(folders, plain_logits, name):
    from cretif_b200.engine import Engine
    from cretif_b200.parts.attention import enable_fused_steps
    eng = Engine(folders[name], dtype="bfloat16", max_tokens=512, step_graphs=False)
    toks = tiny.tokens(name, 40, 7)
    want = plain_logits(name, toks)
    try:
        for on in (True, False):
            enable_fused_steps(on)
            got = run_chunks(eng, toks, [3, 1, 1, 5, 2, 1, 27])
            assert close_routed(got, want, "bfloat16"), (name, on)
    finally:
        enable_fused_steps(True)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_portions_of_a_prompt(engines, plain_logits, name, dtype):
    eng = engines(name, dtype)
    n = LENGTHS[name][-1]
    toks = tiny.tokens(name, n, 3)
    want = plain_logits(name, toks)
    for cuts in ([2, 2, 2, 2], [63, 2, 64], [1, 70, 1, 2], [5] * 12, [n - 2, 2], [16, 1, 15, 1]):
        assert close_routed(run_chunks(eng, toks, cuts), want, dtype), (name, cuts)
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_unequal_batches_against_each_alone_and_reused_slots(engines, plain_logits, name, dtype):
    """Batches of unequal requests on a cache too small for two batches: the second and third
    rounds get slots, blocks, states and saved inputs that were used before."""
    eng = engines(name, dtype, max_tokens=832 if name == "E" else 640)
    lens = LENGTHS[name]
    for round_ in range(3):
        reqs = [tiny.tokens(name, n + 6 + 2 * i, 20 + round_) for i, n in enumerate(lens[:5])]
        prompts = [min(lens[i], len(r)) for i, r in enumerate(reqs)]
        outs = run_batch(eng, reqs, prompts)
        for r, got in zip(reqs, outs):
            assert close_routed(got, plain_logits(name, r), dtype), (name, round_, len(r))
        eng.cache.check()
        assert eng.cache.stats()["slots_live"] == 0
    # a mixture: fresh prompts, further portions and single tokens in the same steps
    reqs = [tiny.tokens(name, n, 30) for n in (40, 9, 27)]
    outs = run_schedule(eng, reqs, [[(0, 18)], [(0, 2), (1, 9)], [(0, 1), (2, 25)],
                                    [(0, 19), (2, 2)]])
    for r, got in zip(reqs, outs):
        assert close_routed(got, plain_logits(name, r), dtype), name
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["B", "E"])
def test_long_decoding(engines, plain_logits, name, dtype):
    """A short prompt and then single tokens over several cache blocks and chunks."""
    eng = engines(name, dtype)
    toks = tiny.tokens(name, 180, 5)
    got = run_tail_by_one(eng, toks, tail=173)
    assert close_routed(got, plain_logits(name, toks), dtype)
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_position_does_not_depend_on_the_cut_or_the_batch(engines, dtype):
    """The same tokens whole, in portions, one by one and beside other requests: the same logits up
    to the order of summation."""
    eng = engines("B", dtype)
    toks = tiny.tokens("B", 150, 9)
    ref = run_whole(eng, toks)
    ways = [run_chunks(eng, toks, [70, 2, 33, 1]), run_tail_by_one(eng, toks, tail=60),
            run_batch(eng, [tiny.tokens("B", 31, 1), toks, tiny.tokens("B", 90, 2)], [9, 100, 64])[1]]
    for got in ways:
        assert rel_err(got, ref) <= (2e-5 if dtype == "float32" else 0.3)
        assert np.abs(got - ref).mean() <= (2e-6 if dtype == "float32" else 1e-2) * np.abs(ref).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_chains_beside_one_another_change_nothing(folders, dtype):
    """Steps of few tokens run the shared expert on a second stream: the same kernels on the same
    inputs, launched or replayed from a graph, and every time the same numbers."""
    from cretif_b200.engine import Engine
    from cretif_b200.parts.side_stream import side_streams_off
    got = {}
    for off in (False, True):
        side_streams_off(off)
        try:
            eng = Engine(folders["A"], dtype=dtype, max_tokens=512)
            got[off] = [run_tail_by_one(eng, tiny.tokens("A", 60, 3), tail=50) for _ in range(3)]
        finally:
            side_streams_off(False)
    for a, b in zip(got[False], got[True]):
        assert rel_err(a, b) < (1e-5 if dtype == "float32" else 2e-2)
    for a in got[False][1:]:
        assert np.array_equal(a, got[False][0])


# ------------------------------------------------------------------ what a position may depend on
def _one_layer_engine(tmp_path_factory, mixer, edit=None, dtype="float32", **options):
    from cretif_b200.engine import Engine
    cfg = tiny.one_layer(mixer, **options)
    d = _write(tmp_path_factory, "edge", cfg, seed=13, edit=edit)
    return Engine(d, dtype=dtype, max_tokens=2048), plain.read_model_folder(d), cfg


def test_a_far_key_among_many(tmp_path_factory):
    """Queries sharpened: most of a row's weight lies on one key, often far back and on the borders of
    the cache's blocks."""
    def sharpen(tensors):
        tensors["l0.mix.q.norm"] = (tensors["l0.mix.q.norm"].float() * 9.0).to(torch.bfloat16)
    for dim in (16, 64):
        for dtype in ("float32", "bfloat16"):
            eng, (pcfg, w), cfg = _one_layer_engine(tmp_path_factory, tiny._att(4, 2, dim, dim, 0.4, 3, 8),
                                                    sharpen, dtype)
            toks = np.random.default_rng(2).integers(0, cfg["vocab"], size=420).tolist()
            want = plain.forward(pcfg, w, toks).numpy()
            assert close(run_whole(eng, toks), want, dtype)
            assert close(run_tail_by_one(eng, toks, tail=50), want, dtype)
            assert close(run_chunks(eng, toks, [127, 2, 64, 130]), want, dtype)


@pytest.mark.parametrize("which, taps", [("attention", 4), ("mamba2", 4), ("attention", 2)])
def test_single_keys_at_block_borders_and_the_first_tokens(tmp_path_factory, which, taps):
    """The last position depends on every earlier token: changing one on a border of the cache's blocks
    or of the chunks, or among the first, moves its logits as it moves the plain model's, and a later
    token moves nothing, to the bit; for a position inside a prompt and for a decoded one."""
    mixer = tiny._att(4, 2, 16, 16, 0.4, taps, 8) if which == "attention" else tiny._ssm(4, 16, 16, 2, 1, taps)

    def keep(tensors):
        if which == "mamba2":              # slow decays: the first tokens still count
            tensors["l0.mix.A_log"] = torch.full_like(tensors["l0.mix.A_log"], -5.0)
    eng, (pcfg, w), cfg = _one_layer_engine(tmp_path_factory, mixer, keep)
    n = 200
    base = np.random.default_rng(taps).integers(0, cfg["vocab"], size=n).tolist()
    want = plain.forward(pcfg, w, base).numpy()
    for run in (run_whole, lambda e, t: run_tail_by_one(e, t, tail=40)):
        ref = run(eng, base)
        assert close(ref, want, "float32")
        for i in (n - 1, n - 60):
            for j in (0, 1, 2, 63, 64, 65, 127, 128, i - taps, i - taps + 1, i - 1, i, i + 1):
                if j >= n:
                    continue
                other = list(base)
                other[j] = (other[j] + 1 + j % 5) % cfg["vocab"]
                row = run(eng, other)[i]
                moved = float(np.abs(row - ref[i]).max())
                if j > i:
                    assert moved == 0.0, (i, j)
                    continue
                by = plain.forward(pcfg, w, other[:i + 1]).numpy()[i] - want[i]
                assert moved > 0.0, (i, j)
                assert np.abs((row - ref[i]) - by).max() <= 1e-4 * np.abs(want).max(), (i, j)


@pytest.mark.parametrize("name", ["A", "B", "D"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens(engines, plain_logits, name, dtype):
    """The convolutions' reach over the start of a sequence, alone and in every portion."""
    eng = engines(name, dtype)
    toks = tiny.tokens(name, 12, 11)
    want = plain_logits(name, toks)
    for cuts in ([1] * 12, [2, 1, 3], [3, 9], [1, 11], [2] * 6):
        assert close_routed(run_chunks(eng, toks, cuts), want, dtype), cuts


def test_memory_of_a_token_far_back(tmp_path_factory):
    """A recurrence that keeps: the first token still shows in the logits hundreds of tokens later,
    across prompt portions and single tokens; and one whose steps wipe the state now and then."""
    def keep(tensors):
        tensors["l0.mix.A_log"] = torch.full_like(tensors["l0.mix.A_log"], -6.0)

    def wild(tensors):
        tensors["l0.mix.A_log"] = torch.tensor([3.0, -3.0]).to(torch.bfloat16)
        rows = tensors["l0.mix.in"].float()
        rows[-2:] *= 12.0
        tensors["l0.mix.in"] = rows.to(torch.bfloat16)
    for edit, far in ((keep, True), (wild, False)):
        eng, (pcfg, w), cfg = _one_layer_engine(tmp_path_factory, tiny._ssm(2, 16, 64, 1, 1, 3), edit)
        n = 300
        base = np.random.default_rng(8).integers(0, cfg["vocab"], size=n).tolist()
        other = [(base[0] + 3) % cfg["vocab"]] + base[1:]
        want, want_other = (plain.forward(pcfg, w, t).numpy() for t in (base, other))
        if far:
            assert np.abs(want[-1] - want_other[-1]).max() > 1e-3 * np.abs(want).max()
        for toks, ref in ((base, want), (other, want_other)):
            assert close(run_whole(eng, toks), ref, "float32")
            assert close(run_chunks(eng, toks, [3, 2, 150, 1, 1, 100]), ref, "float32")
            assert close(run_tail_by_one(eng, toks, tail=60), ref, "float32")


def test_passes_and_their_inputs_count(folders, plain_logits):
    """A pass whose state or keys were shared with another's, an input that is left out and a part of
    the second embedding taken from the wrong layer are other models: the yardstick tells them apart."""
    pcfg, w = plain.read_model_folder(folders["A"])
    toks = tiny.tokens("A", 30, 13)
    want = plain_logits("A", toks)
    for change in ("half", "side", "bias"):
        other = dict(w)
        if change == "half":
            other["loop.in"] = w["loop.in"].clone()
            other["loop.in"][:, 64:] = 0
        elif change == "side":
            other["side.embed"] = torch.roll(w["side.embed"], 8, dims=1)
        else:
            other["l1.norm1.b"] = torch.zeros_like(w["l1.norm1.b"])
        assert rel_err(plain.forward(pcfg, other, toks).numpy(), want) > 20 * TOL["float32"], change


# ------------------------------------------------------------------ generation
@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_entry_point(folders, name):
    """``load(...).generate(...)``: batching, the decode graph (whose warm-up must not advance
    a recurrent state twice) and the run-ahead of the host, against re-running the plain model
    on the growing sequence."""
    import cretif_b200
    eng = cretif_b200.load(folders[name], dtype="float32", max_tokens=2048)
    pcfg, w = plain.read_model_folder(folders[name])
    prompts = [tiny.tokens(name, n, 40) for n in (3, 11, 30)]
    for use_graph in (True, False):
        got = eng.generate(prompts, max_tokens=12, stop_ids=[], use_graph=use_graph)
        for p, r in zip(prompts, got):
            assert len(r.tokens) == 12
            rows = plain.forward(pcfg, w, list(p) + r.tokens[:-1]).numpy()[len(p) - 1:]
            for row, tok in zip(rows, r.tokens):  # every token is the plain model's best, or tied
                assert row.max() - row[tok] <= 1e-4 * np.abs(row).max(), (name, use_graph)
    eng.cache.check()
    assert eng.cache.stats()["slots_live"] == 0


def test_generation_with_more_requests_than_the_cache_holds(folders):
    import cretif_b200
    eng = cretif_b200.load(folders["A"], dtype="bfloat16", max_tokens=256)
    prompts = [tiny.tokens("A", n, 60) for n in (70, 3, 100, 40, 9, 61)]
    together = eng.generate(prompts, max_tokens=9, stop_ids=[])
    assert [len(r.tokens) for r in together] == [9] * 6
    eng.cache.check()
    assert eng.cache.stats()["slots_live"] == 0


def test_the_replay_program_runs_a_pudorax_folder(folders, tmp_path):
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    toks = tiny.tokens("A", 30, 50)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:20], "want": [0, 19]},
                                     {"id": "y", "tokens": toks[:7], "want": [6]}], "end": ["y"]},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[20:21], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[21:22], "want": []}],
              "end": ["x"]}]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model",
                        folders["A"], "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "64"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", text=True,
                       capture_output=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == \
        ["done 0", "done 1", "done 2"]
    cfg, w = plain.read_model_folder(folders["A"])
    want = plain.forward(cfg, w, toks).numpy()
    got0 = np.fromfile(out / "0.f32", dtype="<f4").reshape(3, -1)
    got1 = np.fromfile(out / "1.f32", dtype="<f4").reshape(1, -1)
    assert not (out / "2.f32").exists()
    assert rel_err(got0, want[[0, 19, 6]]) <= 1e-4 and rel_err(got1, want[[20]]) <= 1e-4


def test_the_command_line_writes_and_runs_a_pudorax_folder(tmp_path):
    """``python -m cretif_b200``: a folder with random weights from a config.json, then greedy
    generation from token ids, the same tokens as the entry point gives."""
    import subprocess
    import sys
    import cretif_b200
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg_file = tmp_path / "cfg.json"
    cfg_file.write_text(json.dumps(tiny.P_A))
    folder = str(tmp_path / "model")
    env = dict(os.environ, PYTHONPATH=root)
    r = subprocess.run([sys.executable, "-m", "cretif_b200", folder, "5,6,7,8", "6", "--dtype",
                        "float32", "--random-weights", "21", "--config", str(cfg_file)],
                       capture_output=True, text=True, timeout=600, env=env, cwd=root)
    assert r.returncode == 0, r.stderr[-2000:]
    assert "model: Pudorax" in r.stdout
    line = [l for l in r.stdout.splitlines() if l.startswith("generated ids:")][0]
    got = json.loads(line[len("generated ids:"):line.index("(")].strip())
    eng = cretif_b200.load(folder, dtype="float32", max_tokens=512)
    want = eng.generate([[5, 6, 7, 8]], max_tokens=6, stop_ids=[])[0].tokens
    assert got == want and len(got) == 6
