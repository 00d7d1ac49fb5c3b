"""Gibipel through the engine against the plain implementation (``plain_gibipel``): every
mechanism alone, every way of cutting requests into steps, the edges of windows and pooled blocks,
far keys and far memory, reused slots, greedy generation through the library's own entry point."""
import json
import os

import numpy as np
import pytest
import torch

import gibipel_tiny as tiny
import plain_gibipel as plain
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
           "D": [1, 4, 31, 70, 100], "E": [1, 2, 33, 129, 260]}
WIDE = (".q", ".k", ".v", ".g", ".o", ".i", ".f", ".up", ".gate", ".down")


def _write(tmp_path_factory, name, cfg, seed, edit=None):
    """A model folder for ``cfg`` with seeded random weights; ``edit(tensors)`` may change
    tensors before they are written."""
    from cretif_b200.config import build_gibipel_spec, gibipel_config_from_dict
    from cretif_b200.engine.model import manifest
    from cretif_b200.weights.loader import random_weights, write_model_folder
    d = str(tmp_path_factory.mktemp(f"gibipel_{name}"))
    names, _ = manifest(build_gibipel_spec(gibipel_config_from_dict(cfg)))
    tensors = random_weights(names, seed, torch.bfloat16)
    # wider projections than the default draw: scores and gates that are not all alike
    for k in tensors:
        if k.endswith(WIDE):
            tensors[k] = (tensors[k].float() * 6.0).to(torch.bfloat16)
        elif k in ("embed", "head"):
            tensors[k] = (tensors[k].float() * 20.0).to(torch.bfloat16)
        elif k.endswith((".norm1", ".norm2")):
            tensors[k] = (tensors[k].float() * 0.6).to(torch.bfloat16)
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
    assert arch.name == "Gibipel" and spec.vocab_size == 96 and spec.hidden_size == 64
    eng = Engine(folders["A"], dtype="float32", max_tokens=256)
    groups = eng.cache.stats()["groups"]
    # per layer the window's keys and values, and the entries of its blocks
    assert sorted((g["head_dim"], g["value_dim"], g["window"], g["tokens_per_entry"])
                  for g in groups) == \
        [(16, 8, 0, 5), (16, 8, 21, 1), (16, 24, 0, 4), (16, 24, 9, 1), (24, 24, 0, 13),
         (24, 24, 13, 1)]
    assert eng.cache.stats()["state_bytes"] > 0


# ------------------------------------------------------------------ kernels of the mechanisms
def test_a_factor_on_embedding_and_logits_and_a_norm_of_one_number():
    from cretif_b200.config import PartSpec
    from cretif_b200.csrc import ops
    from cretif_b200.parts import build_part
    g = torch.Generator().manual_seed(1)
    for dt in (torch.float32, torch.bfloat16):
        table = torch.randn(50, 72, generator=g).to(dt)
        ids = torch.tensor([3, 49, 0, 7], dtype=torch.int32)
        out = torch.empty(4, 72, device="cuda")
        fault = torch.zeros(1, dtype=torch.int32, device="cuda")
        ops.embed_rows(table.cuda(), ids.cuda(), out, fault, scale=3.25)
        assert torch.equal(out.cpu(), table[ids.long()].float() * 3.25) and int(fault.item()) == 0
    z = torch.randn(5, 33, generator=g)
    zc = z.cuda()
    ops.scale_in_place(zc, -1.5)
    assert torch.equal(zc.cpu(), z * -1.5)
    norm = build_part("norm", PartSpec("rmsnorm", {"eps": 1e-5, "name": "n", "scalar": True}), 40,
                      torch.float32, "cuda")
    norm.load({"weight": torch.tensor(0.7)})
    h, y = (torch.randn(9, 40, generator=g) for _ in range(2))
    hc = h.cuda()
    norm.add_into(hc, y.cuda())
    want = h.double() + 0.7 * plain.unit(y.double(), 1e-5)
    assert (hc.cpu().double() - want).abs().max() < 1e-5


@pytest.mark.parametrize("R,H", [(1, 2048), (5, 516), (255, 3000), (256, 1024), (3, 4096), (2, 514)])
def test_the_norm_on_an_output_for_few_and_many_rows(R, H):
    from cretif_b200.csrc import ops
    g = torch.Generator().manual_seed(R)
    h, w = torch.randn(R, H, generator=g), torch.randn(H, generator=g)
    for dt in (torch.float32, torch.bfloat16):
        y = (torch.randn(R, H, generator=g) * 3).to(dt)
        want = h.double() + plain.unit(y.double(), 1e-6) * w.double()
        hc, x = h.cuda(), torch.empty(R, H, dtype=torch.bfloat16, device="cuda")
        ops.rmsnorm_add(hc, y.cuda(), w.cuda(), 1e-6, x_out=x)
        assert (hc.cpu().double() - want).abs().max() < 2e-5, dt
        assert torch.equal(x, hc.to(torch.bfloat16))


def test_the_heads_factor_in_every_product():
    """One row, a few rows (the norm in the product's prologue), many rows, and the plain kernels."""
    from cretif_b200.config import PartSpec
    from cretif_b200.parts import build_part
    g = torch.Generator().manual_seed(2)
    H, V = 64, 48
    w = (torch.randn(V, H, generator=g) * 0.2).bfloat16()
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        head = build_part("head", PartSpec("linear_head", {"tied": False, "name": "head", "scale": -0.3,
                                                           "vocab_size": V}), H, dtype, "cuda")
        head.load({"weight": w})
        norm = build_part("norm", PartSpec("rmsnorm", {"eps": 1e-6, "name": "n"}), H, dtype, "cuda")
        norm.load({"weight": torch.ones(H)})
        for R in (1, 7, 200):
            h = torch.randn(R, H, generator=g)
            want = -0.3 * plain.unit(h.double(), 1e-6) @ w.double().T
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


def _pool_for(S, P, G, d, e, dtype):
    from cretif_b200.cache import PoolView
    pk, ptab = _cache_for(max(1, S // P), G, d, dtype)
    pv, _ = _cache_for(max(1, S // P), G, e, dtype)
    return PoolView(pk, pv, ptab, P)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,e,rot,pairing,P", [
    (4, 2, 16, 24, 8, 0, 4), (2, 1, 64, 64, 64, 0, 16), (3, 1, 12, 20, 4, 0, 7),
    (5, 5, 20, 6, 10, 1, 1), (1, 1, 8, 8, 2, 0, 100), (8, 2, 128, 128, 64, 1, 48),
    (2, 2, 16, 16, 0, 0, 3)])
def test_norms_over_whole_projections_rotation_cache_write_and_entries(dtype, H, G, d, e, rot, pairing,
                                                                       P):
    """The kernel between an attention's input product and its scores over a sequence fed in pieces,
    and the entries of the blocks that each piece completes, against the plain functions."""
    from cretif_b200.csrc import ops
    from cretif_b200.parts.position import rotary_table
    g = torch.Generator().manual_seed(4)
    S, base, eps = 300, 300.0, 1e-5
    n_in = (H + G) * d + G * e
    proj = torch.randn(S, n_in + 3, generator=g) * 2
    bias = torch.randn(n_in, generator=g)
    wq, wk = torch.randn(H * d, generator=g), torch.randn(G * d, generator=g)
    sc = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 60.0}
    rows = proj[:, :n_in].double() + bias.double()
    q = (plain.unit(rows[:, :H * d], eps) * wq.double()).reshape(S, H, d)
    k = (plain.unit(rows[:, H * d:(H + G) * d], eps) * wk.double()).reshape(S, G, d)
    v = rows[:, (H + G) * d:].reshape(S, G, e) * -0.7
    cos = sin = None
    if rot:
        cos, sin = rotary_table(base, rot, S, torch.device("cuda"), sc)
        f = plain.frequencies(base, rot, sc)
        if pairing == 0:
            q, k = plain.rotate_front(q, f, rot), plain.rotate_front(k, f, rot)
        else:                        # pair (2i, 2i + 1): the same rotation after a permutation
            perm = list(range(0, rot, 2)) + list(range(1, rot, 2)) + list(range(rot, d))
            inv = np.argsort(perm)
            q = plain.rotate_front(q[..., perm], f, rot)[..., inv]
            k = plain.rotate_front(k[..., perm], f, rot)[..., inv]
    kc, table = _cache_for(S, G, d, dtype)
    vc, _ = _cache_for(S, G, e, dtype)
    pool = _pool_for(S, P, G, d, e, dtype)
    fault = torch.zeros(1, dtype=torch.int32, device="cuda")
    q_out = torch.zeros(S, H * d, dtype=dtype, device="cuda")
    at = 0
    i32 = dict(dtype=torch.int32, device="cuda")
    for n in (1, 2, 30, 1, 1, 1, 1, 200) + (1,) * 63:
        pos, zeros = torch.arange(at, at + n, **i32), torch.zeros(n, **i32)
        args = (proj[at:at + n].cuda(), bias.cuda(), wq.cuda(), wk.cuda(), eps, cos, sin, pairing, rot,
                pos, zeros, zeros[:1], H, G, d, e, q_out[at:at + n])
        ops.projnorm_rope_kv_append(*args, table=table, kc=kc, vc=vc, fault=fault, v_scale=-0.7,
                                    pool=pool if n == 1 else None)
        if n > 1:
            ops.pool_kv(kc, vc, table, pool, torch.tensor([0, n], **i32), torch.tensor([at], **i32),
                        zeros[:1], G, d, e, 64, 1, n, fault)
        at += n
    assert at == S and int(fault.item()) == 0
    tol = 2e-4 if dtype == torch.float32 else 8e-2
    assert (q_out.cpu().double().reshape(S, H, d) - q).abs().max() < tol
    ks, vs = _gather(kc, table, S).double(), _gather(vc, table, S).double()
    assert (ks - k).abs().max() < tol and (vs - v).abs().max() < tol
    # the entries are the means of the rows as the cache holds them, to their own rounding
    etol = 1e-6 if dtype == torch.float32 else 2.0 ** -8
    for cache, stored in ((pool.k, ks), (pool.v, vs)):
        got = _gather(cache, pool.table, S // P).double() if S // P else torch.zeros(0)
        want = plain.block_means(stored, P)
        assert ((got - want).abs() <= etol * want.abs() + 1e-6).all()


def _attention_case(H, G, d, e, window, P, S, seed):
    """Queries, keys and values with a key in seven that stands out: for some queries it is the last
    one their window or a visible block still shows, for others the first one that is not seen."""
    g = torch.Generator().manual_seed(seed)
    q = torch.randn(S, H, d, generator=g)
    k = torch.randn(S, G, d, generator=g)
    q[:, :, 0] += 2.0
    for p in range(S):
        if p % 7 == 3:
            k[p, :, 0] += 3.0
    return q, k, torch.randn(S, G, e, generator=g)


@pytest.mark.parametrize("H,G,d,e,window,P", [
    (4, 2, 64, 64, 70, 16), (2, 1, 128, 128, 64, 64), (8, 2, 32, 32, 65, 8), (3, 3, 16, 16, 129, 5),
    (2, 2, 64, 64, 1, 1), (16, 1, 64, 64, 100, 3), (12, 1, 48, 48, 20, 48), (6, 2, 64, 64, 2, 1),
    (3, 1, 12, 20, 30, 7), (2, 2, 64, 32, 40, 16), (2, 1, 256, 256, 33, 9), (4, 2, 64, 64, 400, 16)])
def test_attention_kernels_with_pooled_entries_and_a_sink(H, G, d, e, window, P):
    """The attention kernels the engine picks (prompt, portion, single tokens, in both element types)
    against the plain softmax over tokens and entries on the same inputs."""
    from cretif_b200.parts.attention import run_attention
    from cretif_b200.parts.base import StepContext
    S = 333
    q, k, v = _attention_case(H, G, d, e, window, P, S, 7)
    sink = torch.randn(H, generator=torch.Generator().manual_seed(3)) * 2
    scale = 0.7 / d ** 0.5
    dev = torch.device("cuda")
    i32 = dict(dtype=torch.int32, device=dev)
    fault = torch.zeros(1, **i32)
    for dtype in (torch.float32, torch.bfloat16):
        qd, kd, vd = (t.to(dtype) for t in (q, k, v))
        kk = torch.cat([kd, plain.block_means(kd.double(), P).to(dtype)]).double()
        vv = torch.cat([vd, plain.block_means(vd.double(), P).to(dtype)]).double()
        visible = torch.cat(plain.window_and_blocks(S, window, P), dim=1)
        want = torch.stack([plain.softmax_with_sink(
            (qd[:, h].double() @ kk[:, h // (H // G)].T) * scale, visible,
            sink[h].double()) @ vv[:, h // (H // G)] for h in range(H)], dim=1).reshape(S, H * e)
        kc, table = _cache_for(S, G, d, dtype)
        vc, _ = _cache_for(S, G, e, dtype)
        t = table[0].cpu()
        for p in range(S):
            kc[t[p // 64], :, p % 64] = kd[p].cuda()
            vc[t[p // 64], :, p % 64] = vd[p].cuda()
        pool = _pool_for(S, P, G, d, e, dtype)
        t = pool.table[0].cpu()
        for b in range(S // P):
            pool.k[t[b // 64], :, b % 64] = kk[S + b].to(dtype).cuda()
            pool.v[t[b // 64], :, b % 64] = vv[S + b].to(dtype).cuda()

        class KV:
            pass
        kv = KV()
        kv.k, kv.v, kv.table, kv.block_tokens, kv.window = kc, vc, table, 64, window

        def ctx(T, first, decode):
            return StepContext(T=T, B=1, tok_ids=torch.zeros(T, **i32),
                               tok_pos=torch.arange(first, first + T, **i32),
                               tok_seq=torch.zeros(T, **i32), seq_slot=torch.zeros(1, **i32),
                               seq_start=torch.tensor([first], **i32),
                               cu_seqlens=torch.tensor([0, T], **i32), is_decode=decode,
                               max_new=T, max_context=512 if decode else first + T, fault=fault,
                               dtype=dtype, device=dev)
        # single tokens where a block has just become visible, and one before
        edge = window + 10 * P - 1 if window + 10 * P < S else S - 2
        for first, T, decode in ((0, S, False), (200, S - 200, False), (130, 2, False),
                                 (S - 1, 1, True), (edge, 1, True), (edge - 1, 1, True),
                                 (0, 1, True), (150, 1, True)):
            out = torch.zeros(T, H * e, dtype=dtype, device=dev)
            run_attention(qd[first:first + T].reshape(T, H * d).cuda(), out,
                          ctx(T, first, decode), kv, H, G, d, scale, window, dtype, sink.cuda(),
                          vd=e, pool=pool)
            err = (out.cpu().double() - want[first:first + T]).abs().max()
            tol = 1e-5 if dtype == torch.float32 else 2e-2
            assert err <= tol * want.abs().max(), (dtype, first, T, decode, float(err))
    assert int(fault.item()) == 0


def _gates(g, S, H, strong):
    """Gate pre-activations; ``strong``: long stretches that forget nothing, sudden resets and loud
    inputs, so that the running maximum is carried far and also overtaken."""
    zi, zf = torch.randn(S, H, generator=g) * 2, torch.randn(S, H, generator=g) * 2 + 3
    if strong:
        zf[:, :] = 9.0
        zf[S // 3::S // 3 + 1] = -8.0
        zi[::17] += 8.0
    return zi, zf


@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("H,d,e", [(2, 128, 128), (3, 32, 64), (1, 64, 16), (5, 16, 48),
                                   (2, 20, 32), (1, 256, 32), (2, 48, 48)])
def test_matrix_memory_in_both_forms(H, d, e, strong):
    """Chunks of 64 tokens and token by token against the recurrence written out, over sequences of
    unequal length fed in pieces that end before, at and after a chunk's edge, with the state
    carried from piece to piece; both forms leave the same state, and other slots alone."""
    from cretif_b200.csrc import ops
    g = torch.Generator().manual_seed(11)
    lens = [331, 64, 129]
    cap, eps, qs = 10.0, 1e-5, d ** -0.5
    bi, bf, nw = torch.randn(H, generator=g), torch.randn(H, generator=g), torch.randn(H * e, generator=g)
    seqs, want = [], []
    for n in lens:
        q, k, v = (torch.randn(n, H * x, generator=g) for x in (d, d, e))
        gate = torch.randn(n, H * e, generator=g)
        zi, zf = _gates(g, n, H, strong)
        seqs.append(torch.cat([q, k, v, gate, zi, zf, torch.full((n, (-2 * H) % 4), float("nan"))], 1))
        li = cap * torch.tanh((zi.double() + bi.double()) / cap)
        lf = plain.log_sigmoid(cap * torch.tanh((zf.double() + bf.double()) / cap))
        o = plain.memory(q.double().reshape(n, H, d) * qs, k.double().reshape(n, H, d),
                         v.double().reshape(n, H, e), li, lf)
        want.append(plain.unit(o, eps).reshape(n, H * e) * nw.double() * torch.sigmoid(gate.double()))
    slots = torch.tensor([3, 0, 2], dtype=torch.int32, device="cuda")
    width = -(-(H * (d * (e + 1) + 1)) // 4) * 4
    states = {}
    for form in ("chunk", "token"):
        state = torch.zeros(5, width, device="cuda")
        state[1] = 7.0
        at = [0, 0, 0]
        for cuts in ((63, 64, 1), (2, 0, 64), (65, 0, 64), (1, 0, 0), (200, 0, 0)):
            live = [i for i, n in enumerate(cuts) if n]
            proj = torch.cat([seqs[i][at[i]:at[i] + cuts[i]] for i in live]).cuda()
            cu = torch.tensor(np.cumsum([0] + [cuts[i] for i in live]), dtype=torch.int32, device="cuda")
            seq = torch.repeat_interleave(torch.arange(len(live), dtype=torch.int32),
                                          torch.tensor([cuts[i] for i in live])).cuda()
            out = torch.full((proj.shape[0], H * e), float("nan"), device="cuda")
            ops.matrix_memory(proj, bi.cuda(), bf.cuda(), cap, qs, state, cu, slots[live].contiguous(),
                              seq, len(live), H, d, e, nw.cuda(), eps, out, form=form)
            row = 0
            for i in live:
                got = out[row:row + cuts[i]].cpu().double()
                ref = want[i][at[i]:at[i] + cuts[i]]
                # a read-out that is a small difference of large terms is normed up with its
                # rounding: a few parts in a thousand on single elements, nothing on average
                diff = (got - ref).abs()
                assert diff.max() <= 5e-3 and diff.mean() <= 1e-5, (form, cuts, i, float(diff.max()))
                row += cuts[i]
                at[i] += cuts[i]
        assert at == lens
        assert bool((state[1] == 7.0).all()) and bool((state[4] == 0.0).all())
        states[form] = state
    diff = (states["chunk"] - states["token"]).abs().max()
    assert diff <= 5e-5 * max(1.0, float(states["token"].abs().max())), float(diff)


def test_matrix_memory_options_and_refusals():
    from cretif_b200.csrc import ops
    H, d, e, T = 2, 6, 16, 70
    g = torch.Generator().manual_seed(5)
    proj = torch.randn(T, 2 * H * (d + e) + 2 * H, generator=g).cuda()
    zero = torch.zeros(H, device="cuda")
    i32 = dict(dtype=torch.int32, device="cuda")
    state = torch.randn(1, H * (d * (e + 1) + 1), generator=g).cuda()
    before = state.clone()
    out = torch.empty(T, H * e, device="cuda")
    args = (proj, zero, zero, 5.0, 1.0, state, torch.tensor([0, T], **i32), torch.zeros(1, **i32),
            torch.zeros(T, **i32), 1, H, d, e, torch.ones(H * e, device="cuda"), 1e-5, out)
    with pytest.raises(ops.KernelError):
        ops.matrix_memory(*args, form="chunk")                # d is no multiple of four
    ops.matrix_memory(*args, form="auto", write_state=False)  # takes the other form
    assert torch.equal(state, before) and bool(torch.isfinite(out).all())
    ops.matrix_memory(*args, form="token")
    assert not torch.equal(state, before)


def test_matrix_memory_of_many_sequences_of_one_token():
    from cretif_b200.csrc import ops
    g = torch.Generator().manual_seed(8)
    H, d, e, B, steps, cap = 3, 32, 16, 21, 9, 6.0
    width = -(-(H * (d * (e + 1) + 1)) // 4) * 4
    bi, bf = torch.randn(H, generator=g), torch.randn(H, generator=g) + 2
    rows = torch.randn(steps, B, 2 * H * (d + e) + 2 * H, generator=g)
    slots = torch.randperm(30, generator=g)[:B].to(torch.int32).cuda()
    state = torch.zeros(30, width, device="cuda")
    i32 = dict(dtype=torch.int32, device="cuda")
    got = []
    for s in range(steps):
        out = torch.empty(B, H * e, device="cuda")
        ops.matrix_memory(rows[s].cuda(), bi.cuda(), bf.cuda(), cap, 0.5, state, torch.arange(B + 1, **i32),
                          slots, torch.arange(B, **i32), B, H, d, e, torch.ones(H * e, device="cuda"),
                          1e-5, out)
        got.append(out.cpu())
    got = torch.stack(got)
    for b in (0, 7, B - 1):
        r = rows[:, b].double()
        q, k = (r[:, x * H * d:(x + 1) * H * d].reshape(steps, H, d) for x in (0, 1))
        v = r[:, 2 * H * d:2 * H * d + H * e].reshape(steps, H, e)
        gate = r[:, 2 * H * d + H * e:2 * H * (d + e)]
        li = cap * torch.tanh((r[:, -2 * H:-H] + bi.double()) / cap)
        lf = plain.log_sigmoid(cap * torch.tanh((r[:, -H:] + bf.double()) / cap))
        want = plain.unit(plain.memory(q * 0.5, k, v, li, lf), 1e-5).reshape(steps, H * e) \
            * torch.sigmoid(gate)
        assert (got[:, b].double() - want).abs().max() < 2e-3, b


@pytest.mark.parametrize("E,top,groups,keep", [(20, 4, 4, 3), (8, 2, 4, 2), (6, 3, 2, 2), (4, 2, 4, 3),
                                               (3, 1, 0, 0), (1, 1, 1, 1), (64, 6, 8, 3),
                                               (256, 8, 16, 4), (40, 5, 0, 0)])
def test_routing_by_softmax_with_a_correction_and_best_of_group(E, top, groups, keep):
    """``shift``: a correction that pushes every choice score below zero, so that anything left out
    by its group and counted as zero would win."""
    from cretif_b200.csrc import ops
    g = torch.Generator().manual_seed(E + top)
    T, H = 70, 48
    x = torch.randn(T, H, generator=g)
    router = torch.randn(E, H, generator=g) * 0.4
    for shift in (0.0, -3.0):
        corr = torch.randn(E, generator=g) * 0.1 + shift
        scores = torch.softmax(x.double() @ router.double().T, dim=-1)
        for way in ("route", "topk"):
            ids = torch.zeros(T, top, dtype=torch.int32, device="cuda")
            wts = torch.zeros(T, top, dtype=torch.float32, device="cuda")
            rule = dict(renorm=True, groups=groups, keep=keep, sum_eps=1e-20, softmax=True,
                        group_best=True, correction=corr.cuda())
            if way == "route":
                ops.moe_route(x.cuda(), router.cuda(), top, ids, wts, **rule)
            else:
                ops.moe_topk((x.double() @ router.double().T).float().cuda(), top, ids, wts, **rule)
            for t in range(T):
                want = plain.choose(scores[t], corr.double(), top,
                                    {"count": groups, "keep": keep} if groups else None)
                w = scores[t][want] / scores[t][want].sum()
                got = dict(zip(ids[t].tolist(), wts[t].tolist()))
                assert set(got) == set(want), (way, t, shift)
                assert all(abs(got[e] - float(b)) < 1e-5 for e, b in zip(want, w)), (way, t)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mlp", [tiny._moe(6, 2, 64, identity=2, groups=(4, 2), shared=32),
                                 tiny._moe(10, 3, 40, identity=6, shared=64),
                                 tiny._moe(4, 2, 64), tiny._moe(2, 4, 24, identity=3)])
def test_experts_through_every_product(tmp_path_factory, mlp, dtype):
    """A handful of pairs, sorted pairs and (in bfloat16) whole tiles on the tensor cores; tokens all
    of whose choices are identities among them."""
    from cretif_b200.csrc import ops
    from cretif_b200.engine import Engine
    from cretif_b200.parts.experts import few_pairs_off

    def edit(tensors):
        # (scores far apart: no choice is a close call)
        tensors["l0.mlp.router"] = (tensors["l0.mlp.router"].float() * 2).to(torch.bfloat16)
    cfg = tiny.one_layer("both", mlp=mlp, width=64)
    d = _write(tmp_path_factory, "experts", cfg, seed=5, edit=edit)
    eng = Engine(d, dtype=dtype, max_tokens=1024, step_graphs=False)
    pcfg, w = plain.read_model_folder(d)
    toks = np.random.default_rng(6).integers(0, cfg["vocab"], size=150).tolist()
    want = plain.forward(pcfg, w, toks).numpy()
    if mlp["router"].get("identity"):
        # the identities count: without them the logits are others
        other = dict(w)
        other["l0.mlp.correction"] = w["l0.mlp.correction"].clone()
        other["l0.mlp.correction"][mlp["router"]["experts"]:] -= 1e3
        if mlp["router"]["experts"] >= mlp["router"]["top"] and "groups" not in mlp["router"]:
            assert rel_err(plain.forward(pcfg, other, toks).numpy(), want) > 0.02
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


# ------------------------------------------------------------------ each mixer alone in a model
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("side", ["left", "right", "both"])
def test_one_layer_of_each_mixer(tmp_path_factory, side, dtype):
    from cretif_b200.engine import Engine
    cfg = tiny.one_layer(side)
    d = _write(tmp_path_factory, "one_" + side, cfg, seed=9)
    eng = Engine(d, dtype=dtype, max_tokens=1024)
    pcfg, w = plain.read_model_folder(d)
    rng = np.random.default_rng(3)
    for n in (1, 2, 13, 90):
        toks = rng.integers(0, cfg["vocab"], size=n).tolist()
        want = plain.forward(pcfg, w, toks).numpy()
        assert close(run_whole(eng, toks), want, dtype), (side, n)
        assert close(run_tail_by_one(eng, toks, tail=n), want, dtype), (side, n)
        assert close(run_chunks(eng, toks, [2, 5, 2, 30]), want, dtype), (side, n)
    eng.cache.check()


@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_sides_together_and_apart(folders, plain_logits, name):
    """The sides' shared products against each side through its own forward."""
    from cretif_b200.engine import Engine
    from cretif_b200.parts.parallel import sides_apart
    for dtype in ("float32", "bfloat16"):
        eng = Engine(folders[name], dtype=dtype, max_tokens=512, step_graphs=False)
        toks = tiny.tokens(name, 90, 8)
        want = plain_logits(name, toks)
        got = {}
        for apart in (False, True):
            try:
                sides_apart(apart)
                got[apart] = run_chunks(eng, toks, [40, 1, 1, 20, 2])
            finally:
                sides_apart(False)
            assert close_routed(got[apart], want, dtype), (name, apart)
        assert rel_err(got[True], got[False]) < (1e-4 if dtype == "float32" else 0.3)


def test_mixers_that_cannot_share_products_run_one_after_the_other():
    """Any mixer can stand beside another: two attentions without the head-by-head kernel, each with
    keys and values of its own."""
    from cretif_b200.config import BranchSpec, LayerSpec, ModelSpec, PartSpec, ScheduleEntry
    from cretif_b200.cache import SequenceCache
    from cretif_b200.engine.model import Model, manifest
    from cretif_b200.parts.base import StepContext
    from cretif_b200.weights.loader import random_weights

    def att(window):
        return {"num_heads": 2, "num_kv_heads": 1, "head_dim": 16, "scale": 0.25, "window": window,
                "position": {"kind": "rotary", "theta": 100.0, "rotary_dim": 16}}

    def spec(mixer):
        return ModelSpec("x", 40, 32, PartSpec("token_embedding", {"name": "embed"}),
                         [LayerSpec("l.", (BranchSpec("mixer", mixer),))], [ScheduleEntry(0)],
                         PartSpec("rmsnorm", {"eps": 1e-5, "name": "n"}),
                         PartSpec("linear_head", {"tied": True, "tied_to": "embed"}), 256)

    def names(p):
        return {"names": {k: p + k for k in "qkvo"}}
    both = PartSpec("parallel", {"sides": [
        {"name": "a", "kind": "attention", "params": {**att(0), **names("a.")}, "scale": 0.5},
        {"name": "b", "kind": "attention", "params": {**att(7), **names("b.")}, "scale": -2.0}]})
    man, _ = manifest(spec(both))
    w = random_weights(man, 3, torch.bfloat16)
    w = {k: (v.float() * (4.0 if k.startswith("l.") else 1.0)).to(torch.bfloat16) for k, v in w.items()}
    ids = torch.randint(0, 40, (30,), generator=torch.Generator().manual_seed(1), dtype=torch.int32)
    i32 = dict(dtype=torch.int32, device="cuda")

    def run(mixer, prefix):
        m = Model(spec(mixer), torch.float32, "cuda")
        m.load({k: w[prefix(k)] for k in manifest(spec(mixer))[0]})
        cache = SequenceCache(m.cache_requests(), 256, torch.float32, "cuda", max_len=128)
        m.prepare(128)
        s = cache.alloc_slot()
        cache.begin_step([(s, 30)])
        ctx = StepContext(T=30, B=1, tok_ids=ids.cuda(), tok_pos=torch.arange(30, **i32),
                          tok_seq=torch.zeros(30, **i32), seq_slot=torch.tensor([s], **i32),
                          seq_start=torch.zeros(1, **i32), cu_seqlens=torch.tensor([0, 30], **i32),
                          is_decode=False, max_new=30, max_context=30,
                          fault=torch.zeros(1, **i32), dtype=torch.float32, device=torch.device("cuda"))
        streams = []
        ctx.extras["streams"] = streams
        m.forward(ctx, cache, None)
        return streams[0].cpu(), w["embed"][ids.long()].float()
    got, h = run(both, lambda k: k)
    one = {}
    for p, window in (("a.", 0), ("b.", 7)):
        alone, _ = run(PartSpec("attention", {**att(window), **names(p)}), lambda k: k)
        one[p] = alone - h
    want = 0.5 * one["a."] - 2.0 * one["b."]
    assert (got - h - want).abs().max() < 1e-5 * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("name", ["A", "B", "D", "E"])
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
    got = {}
    try:
        for on in (True, False):
            enable_fused_steps(on)
            got[on] = run_chunks(eng, toks, [3, 1, 1, 5, 2, 1, 27])
            assert close_routed(got[on], want, "bfloat16"), (name, on)
    finally:
        enable_fused_steps(True)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("graphs", [False, True])
def test_chains_beside_one_another_change_nothing(folders, dtype, graphs):
    """Steps of few tokens fork onto a second stream (the sides of a mixer, a shared expert): the same
    kernels on the same inputs, launched or replayed from a graph, and every time the same numbers."""
    from cretif_b200.engine import Engine
    from cretif_b200.parts.side_stream import side_streams_off
    got = {}
    for off in (False, True):
        side_streams_off(off)
        try:
            eng = Engine(folders["A"], dtype=dtype, max_tokens=512, step_graphs=graphs)
            got[off] = [run_tail_by_one(eng, tiny.tokens("A", 60, 3), tail=50) for _ in range(3)]
            got[off] += run_batch(eng, [tiny.tokens("A", n, 4) for n in (30, 22, 9)], [4, 8, 2])
        finally:
            side_streams_off(False)
    if dtype == "bfloat16":
        for a, b in zip(got[False], got[True]):
            assert rel_err(a, b) < 1e-2           # (the shared expert joins the sum at another place)
    else:
        for a, b in zip(got[False], got[True]):
            assert rel_err(a, b) < 1e-5
    for a in got[False][1:3]:
        assert np.array_equal(a, got[False][0])   # and every time the same


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
    rounds get slots, blocks, entries and states that were used before."""
    eng = engines(name, dtype, max_tokens=960 if name == "E" else 640)
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
def test_long_decoding_past_every_window(engines, plain_logits, name, dtype):
    """A short prompt and then single tokens: every window passes over decoded tokens, every kind of
    block is completed and becomes visible while decoding, and window blocks are given back."""
    eng = engines(name, dtype)
    toks = tiny.tokens(name, 240, 5)
    got = run_tail_by_one(eng, toks, tail=230)
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


# ------------------------------------------------------------------ what a position may depend on
def _one_layer_engine(tmp_path_factory, side, mixer=None, edit=None, dtype="float32"):
    from cretif_b200.engine import Engine
    cfg = tiny.one_layer(side, mixer)
    d = _write(tmp_path_factory, f"edge_{side}", cfg, seed=13, edit=edit)
    return Engine(d, dtype=dtype, max_tokens=2048), plain.read_model_folder(d), cfg


def _sees(i, j, window, P):
    return 0 <= i - j < window or (j // P) * P + P - 1 <= i - window


@pytest.mark.parametrize("window,P", [(1, 1), (7, 4), (64, 16), (65, 8), (129, 5), (20, 48), (3, 1)])
def test_a_window_and_its_blocks_end_where_they_should(tmp_path_factory, window, P):
    """One layer whose matrix memory counts nothing: the logits at position i depend on the tokens of
    its window and of the blocks wholly before it, and on nothing else.  Changing the token on one side
    of each edge changes them, on the other side it does not, for a position inside a prompt and
    for a decoded one."""
    mixer = tiny._mixer(tiny._left(4, 2, 16, 16, window, P, 0.4, 8), tiny._right(2, 16, 16), 1.0, 0.0)
    eng, (pcfg, w), cfg = _one_layer_engine(tmp_path_factory, "left", mixer)
    rng = np.random.default_rng(window)
    n = window + 3 * P + 70
    base = rng.integers(0, cfg["vocab"], size=n).tolist()
    want = plain.forward(pcfg, w, base).numpy()
    for run in (run_whole, lambda e, t: run_tail_by_one(e, t, tail=40)):
        ref = run(eng, base)
        assert close(ref, want, "float32")
        for i in (n - 1, n - 18):
            out = i - window                              # the token that has just left the window
            last_block = (i - window + 1) // P * P        # the first token no visible block holds
            places = {i - window + 1, out, last_block, last_block - 1, last_block - P, 0}
            for j in sorted(p for p in places if 0 <= p <= i):
                seen = _sees(i, j, window, P)
                other = list(base)
                other[j] = (other[j] + 1 + j % 5) % cfg["vocab"]
                moved = float(np.abs(run(eng, other)[i] - ref[i]).max())
                # what is not seen changes nothing of position i's arithmetic at all
                assert (moved > 1e-7) if seen else (moved == 0.0), (window, P, i, j, seen, moved)
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_edges_in_the_fast_kernels(tmp_path_factory, dtype):
    """Heads of 64 (the tensor-core kernels in bfloat16): the same dependence, with the query norm's
    weight raised so that single keys carry the rows."""
    def sharpen(tensors):
        tensors["l0.mix.left.q.norm"] = (tensors["l0.mix.left.q.norm"].float() * 5.0).to(torch.bfloat16)
    window, P = 100, 6
    mixer = tiny._mixer(tiny._left(4, 2, 64, 64, window, P, 0.2, 32, 5000.0), tiny._right(2, 16, 16),
                        1.0, 0.0)
    eng, (pcfg, w), cfg = _one_layer_engine(tmp_path_factory, "left", mixer, sharpen, dtype)
    rng = np.random.default_rng(4)
    n = 300
    base = rng.integers(0, cfg["vocab"], size=n).tolist()
    want = plain.forward(pcfg, w, base).numpy()
    for run in (run_whole, lambda e, t: run_tail_by_one(e, t, tail=40),
                lambda e, t: run_chunks(e, t, [130, 2, 70])):
        ref = run(eng, base)
        assert close(ref, want, dtype)
        for i in (n - 1, n - 31):
            last_block = (i - window + 1) // P * P
            for j in (i - window + 1, last_block, last_block - 1, last_block - P):
                seen = _sees(i, j, window, P)
                best, other = -1.0, None
                for c in range(1, 8):
                    cand = list(base)
                    cand[j] = (base[j] + 11 * c) % cfg["vocab"]
                    by = float(np.abs(plain.forward(pcfg, w, cand).numpy()[i] - want[i]).max()) \
                        if seen else 0.0
                    if by > best:
                        best, other = by, cand
                moved = float(np.abs(run(eng, other)[i] - ref[i]).max())
                if not seen:
                    assert moved == 0.0, (dtype, i, j, moved)
                elif dtype == "float32":
                    assert abs(moved - best) <= 1e-3 * np.abs(want).max() and best > 0, (i, j, moved, best)
                elif best > 0.05 * np.abs(want).max():
                    assert moved > 0.2 * best, (i, j, moved, best)


def test_a_far_block_among_many(tmp_path_factory):
    """Queries sharpened: most of a row's weight lies on one entry or key, often far back and beyond
    block borders of both caches."""
    def sharpen(tensors):
        tensors["l0.mix.left.q.norm"] = (tensors["l0.mix.left.q.norm"].float() * 9.0).to(torch.bfloat16)
    for dim, P in ((16, 3), (64, 2)):
        mixer = tiny._mixer(tiny._left(4, 2, dim, dim, 40, P, 0.4, 8), tiny._right(2, 16, 16), 1.0, 0.0)
        for dtype in ("float32", "bfloat16"):
            eng, (pcfg, w), cfg = _one_layer_engine(tmp_path_factory, "left", mixer, sharpen, dtype)
            toks = np.random.default_rng(2).integers(0, cfg["vocab"], size=420).tolist()
            want = plain.forward(pcfg, w, toks).numpy()
            assert close(run_whole(eng, toks), want, dtype)
            assert close(run_tail_by_one(eng, toks, tail=50), want, dtype)


def test_loud_sinks(tmp_path_factory):
    def edit(tensors):
        tensors["l0.mix.left.sink"] = torch.tensor([4.0, -4.0, 2.0, 0.5]).to(torch.bfloat16)
    for dim in (16, 64):
        mixer = tiny._mixer(tiny._left(4, 2, dim, dim, 40, 8, 0.3, 8), tiny._right(2, 16, 16), 1.0, 0.0)
        for dtype in ("float32", "bfloat16"):
            eng, (pcfg, w), cfg = _one_layer_engine(tmp_path_factory, "left", mixer, edit, dtype)
            toks = np.random.default_rng(5).integers(0, cfg["vocab"], size=120).tolist()
            want = plain.forward(pcfg, w, toks).numpy()
            assert close(run_whole(eng, toks), want, dtype)
            assert close(run_tail_by_one(eng, toks, tail=30), want, dtype)
            w2 = dict(w)
            w2["l0.mix.left.sink"] = torch.full_like(w["l0.mix.left.sink"], -30.0)
            assert rel_err(plain.forward(pcfg, w2, toks).numpy(), want) > 0.02


def test_memory_of_a_token_far_back(tmp_path_factory):
    """A matrix memory alone whose forget gates are open: the first token still shows in the logits
    hundreds of tokens later, across prompt portions and single tokens, and with gates that shut now
    and then the running maximum is carried and overtaken as in the recurrence written out."""
    def keep(tensors):
        tensors["l0.mix.right.f.b"] = torch.full_like(tensors["l0.mix.right.f.b"], 8.0)
        tensors["l0.mix.right.f"] = (tensors["l0.mix.right.f"].float() * 0.1).to(torch.bfloat16)

    def wild(tensors):
        for k in ("f", "i"):
            tensors[f"l0.mix.right.{k}"] = (tensors[f"l0.mix.right.{k}"].float() * 8.0).to(torch.bfloat16)
    for edit, far in ((keep, True), (wild, False)):
        mixer = tiny._mixer(tiny._left(2, 1, 8, 8, 4, 2, 0.4, 8), tiny._right(2, 64, 16, 12.0), 0.0, 1.0)
        eng, (pcfg, w), cfg = _one_layer_engine(tmp_path_factory, "right", mixer, edit)
        rng = np.random.default_rng(8)
        n = 300
        base = rng.integers(0, cfg["vocab"], size=n).tolist()
        other = [(base[0] + 3) % cfg["vocab"]] + base[1:]
        want, want_other = (plain.forward(pcfg, w, t).numpy() for t in (base, other))
        if far:
            assert np.abs(want[-1] - want_other[-1]).max() > 1e-3 * np.abs(want).max()
        for toks, ref in ((base, want), (other, want_other)):
            assert close(run_whole(eng, toks), ref, "float32")
            assert close(run_chunks(eng, toks, [3, 2, 150, 1, 1, 100]), ref, "float32")
            assert close(run_tail_by_one(eng, toks, tail=60), ref, "float32")


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
        got = eng.generate(prompts, max_tokens=14, stop_ids=[], use_graph=use_graph)
        for p, r in zip(prompts, got):
            seq = list(p)
            for tok in r.tokens:        # every token is the plain model's best, or tied with it
                row = plain.forward(pcfg, w, seq)[-1].numpy()
                assert row.max() - row[tok] <= 1e-4 * np.abs(row).max(), (name, use_graph)
                seq.append(tok)
            assert len(r.tokens) == 14
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


def test_the_replay_program_runs_a_gibipel_folder(folders, tmp_path):
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


def test_the_command_line_writes_and_runs_a_gibipel_folder(tmp_path):
    """``python -m cretif_b200``: a folder with random weights from a config.json, then greedy
    generation from token ids, the same tokens as the entry point gives."""
    import subprocess
    import sys
    import cretif_b200
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg_file = tmp_path / "cfg.json"
    cfg_file.write_text(json.dumps(tiny.G_A))
    folder = str(tmp_path / "model")
    env = dict(os.environ, PYTHONPATH=root)
    r = subprocess.run([sys.executable, "-m", "cretif_b200", folder, "5,6,7,8", "6", "--dtype",
                        "float32", "--random-weights", "21", "--config", str(cfg_file)],
                       capture_output=True, text=True, timeout=600, env=env, cwd=root)
    assert r.returncode == 0, r.stderr[-2000:]
    assert "model: Gibipel" in r.stdout
    line = [l for l in r.stdout.splitlines() if l.startswith("generated ids:")][0]
    got = json.loads(line[len("generated ids:"):line.index("(")].strip())
    eng = cretif_b200.load(folder, dtype="float32", max_tokens=512)
    want = eng.generate([[5, 6, 7, 8]], max_tokens=6, stop_ids=[])[0].tokens
    assert got == want and len(got) == 6
