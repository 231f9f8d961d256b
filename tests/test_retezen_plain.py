"""The Retezen decoder without a GPU: its configuration and plan, what the cache manager does with a window whose blocks are
pooled (pages of an incomplete block that the window has passed, pages of rows that stand for several tokens), and a
second reading of every function of the plain implementation, element by element with ``math`` alone."""

import copy
import math
import random

import pytest
import torch

import plain_retezen as plain
import retezen_cases as cases
from ferrisinfer_b200.cache.manager import CacheManager
from ferrisinfer_b200.config import resolve_config
from ferrisinfer_b200.errors import ConfigError, OutOfPages, UnsupportedError, WeightLoadError
from ferrisinfer_b200.parts import build_model
from ferrisinfer_b200.parts.attention import GroupedQueryAttention
from ferrisinfer_b200.parts.base import CombinedNeed, PagedKV
from ferrisinfer_b200.parts.feed_forward import MixtureOfExperts
from ferrisinfer_b200.parts.plan import PartSpec
from ferrisinfer_b200.weights.loader import check_tensors

F64 = torch.float64


# ------------------------------------------------------------------------------------------ configuration, plan
@pytest.mark.parametrize("case", sorted(cases.CASES))
def test_configuration_round_trip_and_tensor_names(case):
    cfg = cases.CASES[case]
    arch, c = resolve_config(copy.deepcopy(cfg))
    assert arch.name == "Retezen" and c.to_dict() == cfg
    model = build_model(arch.plan(c))
    specs = model.tensor_specs()
    shapes = cases.tensor_shapes(cfg)
    assert {s.name: tuple(s.shape) for s in specs if s.name in shapes} == shapes
    first = [i for i, e in enumerate(cfg["layers"]) if e["mixer"]["v_mix"]][:1]
    unused = {f"l{i}.mix.vmix" for i in first}  # the source of the values mixes nothing itself
    required = {s.name for s in specs if s.required}
    assert required == set(shapes) - unused
    check_tensors(specs, shapes, model.plan.extra["ignorable_tensors"])
    missing = {n: s for n, s in shapes.items() if n not in unused}
    check_tensors(specs, missing, model.plan.extra["ignorable_tensors"])
    with pytest.raises(WeightLoadError):
        check_tensors(specs, {n: s for n, s in shapes.items() if n != "pos"})
    assert model.plan.max_positions == cfg["max_positions"] and model.plan.positions_bounded


def test_absent_keys():
    cfg = copy.deepcopy(cases.CASE_D)
    del cfg["logit_scale"]
    for e in cfg["layers"]:
        del e["mixer"]["v_mix"]
    del cfg["layers"][0]["mixer"]["kv_heads"], cfg["layers"][0]["mixer"]["vdim"], cfg["layers"][1]["mixer"]["mask"]["pool"]
    cfg["layers"][1]["mlp"] = None
    _, c = resolve_config(cfg)
    assert c.logit_scale == 1.0 and not any(x.mixer.v_mix for x in c.layers)
    assert c.layers[0].mixer.kv_heads == 2 and c.layers[0].mixer.vdim == 128
    assert c.layers[1].mixer.pool is None and c.layers[1].mixer.window == 16 and c.layers[1].mlp is None


@pytest.mark.parametrize("change,error", [
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), ConfigError),
    (lambda d: d["layers"][0]["mixer"].update(vdim=25), ConfigError),  # the mixing layers' values no longer match
    (lambda d: d["layers"][0]["mixer"]["mask"].update(pool=0), ConfigError),
    (lambda d: d["layers"][0]["mixer"]["mask"].pop("size"), ConfigError),
    (lambda d: d["layers"][0]["mixer"].update(v_mix="yes"), ConfigError),
    (lambda d: d["layers"][0]["mlp"].update(limit=0.0), ConfigError),
    (lambda d: d["layers"][1]["mlp"]["router"].update(top=7), ConfigError),
    (lambda d: d["layers"][1]["mlp"].update(kind="shared"), UnsupportedError),
    (lambda d: d["layers"][2].update(type="recurrent"), UnsupportedError),
    (lambda d: d.pop("max_positions"), ConfigError),
])
def test_configuration_errors(change, error):
    bad = copy.deepcopy(cases.CASE_A)
    change(bad)
    with pytest.raises(error):
        resolve_config(bad)


def test_parts_refuse_what_does_not_go_together():
    base = dict(hidden_size=32, num_heads=2, num_kv_heads=1, head_dim=16, qk_norm={"eps": 1e-6},
                tensor_names={n: n for n in "qkvo"})
    with pytest.raises(ValueError):  # blocks stand before a window
        GroupedQueryAttention(position=PartSpec("none"), pool=4, **base)
    with pytest.raises(ValueError):  # a block has no distance of its own
        GroupedQueryAttention(position=PartSpec("distance_slopes", {"span": 8.0}), window=8, pool=4, **base)
    with pytest.raises(ValueError):
        GroupedQueryAttention(position=PartSpec("none"), value_mix={"lambda": "vmix", "role": "third"}, **base)
    with pytest.raises(ValueError):
        MixtureOfExperts(32, 16, 4, 2, sigmoid_scores=True, scored={"groups": 1, "keep": 1})
    with pytest.raises(ValueError):
        MixtureOfExperts(32, 16, 4, 2, input_weights=True, identity=1, scored={"groups": 1, "keep": 1})


def test_cache_needs_by_mask():
    arch, c = resolve_config(cases.CASE_B)
    needs = build_model(arch.plan(c)).cache_needs()
    assert needs[0] == PagedKV(1, 40, 21, 24) and needs[1] == PagedKV(2, 16, None, 20)
    assert needs[2] == CombinedNeed((PagedKV(4, 24, 33, 10, run=7), PagedKV(4, 24, None, 10, stride=7)))
    assert needs[3] == CombinedNeed((PagedKV(1, 64, 9, run=4), PagedKV(1, 64, stride=4)))


# ------------------------------------------------------------------------------------------ the cache manager
@pytest.mark.parametrize("window,pool,page", [(24, 5, 16), (5, 16, 16), (7, 40, 16), (1, 3, 4), (33, 1, 8), (16, 16, 16)])
def test_pages_of_a_window_with_pooled_blocks(window, pool, page):
    """Steps of changing size: every key that a token of the step reads and every key of a block that the step completes has
    a page, every block that a token may read has a row, and after the step no page is held that nothing needs any more."""
    need = CombinedNeed((PagedKV(2, 8, window, run=pool), PagedKV(2, 8, stride=pool)))
    mgr = CacheManager([need], page, 64, 2)
    mgr.admit("a")
    rng = random.Random(window * 1000 + pool * 10 + page)
    total = 0
    while total < 4 * max(window, pool) + 40:
        n = rng.choice([1, 1, 2, 3, window // 2 + 1, window + 3, pool])
        before, total = total, total + n
        mgr.extend("a", total)
        tokens, means = mgr.block_table("a", 0), mgr.block_table("a", 1)
        for p in range(before, total):
            assert all(tokens[j // page] >= 0 for j in range(max(0, p - window + 1), p + 1))
            if (p + 1) % pool == 0:  # the block that p completes
                assert all(tokens[j // page] >= 0 for j in range(p + 1 - pool, p + 1)), (p, before)
                assert means[(p // pool) // page] >= 0
            assert all(means[b // page] >= 0 for b in range(max(0, p - window + 1) // pool))
        mgr.commit("a", total)
        tokens = mgr.block_table("a", 0)
        first = min(max(0, total - window + 1), total - total % pool) // page
        assert all(b < 0 for b in tokens[:first]) and all(b >= 0 for b in tokens[first:])
        assert len(mgr.block_table("a", 1)) == -(-(total // pool) // page)
        mgr.check_invariants()
    held = sum(1 for b in mgr.block_table("a", 0) if b >= 0)
    assert held <= -(-max(window, pool) // page) + 1
    mgr.release("a")
    assert all(g.pool.num_used == 0 for g in mgr.groups)


def test_pools_of_rows_for_several_tokens_are_sized_by_the_tokens_and_always_suffice():
    """However the tokens that the pool was made for are divided among the requests, the pooled rows fit."""
    rng = random.Random(3)
    for page, pages, requests, pool in ((16, 72, 4, 12), (16, 9, 4, 3), (4, 30, 3, 1), (16, 6, 2, 200)):
        mgr = CacheManager([CombinedNeed((PagedKV(1, 4, 20, run=pool), PagedKV(1, 4, stride=pool)))], page, pages, requests)
        want = pages if pool == 1 else min(pages, -(-pages // pool) + requests)
        assert mgr.groups[1].pool.num_pages == want
        for _ in range(20):
            left = pages
            for r in range(requests):
                take = left if r == requests - 1 else rng.randint(0, left)
                left -= take
                mgr.admit(r)
                total = 0
                while total < take * page:
                    total = min(take * page, total + rng.randint(1, 3 * page))
                    mgr.extend(r, total)
                    mgr.commit(r, total)
            mgr.check_invariants()
            for r in range(requests):
                mgr.release(r)
            assert all(g.pool.num_used == 0 for g in mgr.groups)


def test_a_step_that_the_pooled_rows_do_not_fit_takes_nothing():
    mgr = CacheManager([CombinedNeed((PagedKV(1, 4, 8, run=4), PagedKV(1, 4, stride=4)))], 4, {0: 100, 1: 1}, 2)
    mgr.admit("a")
    mgr.extend("a", 19)  # four rows: one page
    with pytest.raises(OutOfPages):
        mgr.extend("a", 20)
    assert len(mgr.block_table("a", 0)) == 5 and len(mgr.block_table("a", 1)) == 1
    mgr.release("a")


def test_prompts_are_not_shared_where_rows_stand_for_several_tokens():
    assert CacheManager([PagedKV(1, 4, stride=4)], 4, 8, 2, prefix_sharing=True).prefix is None
    assert CacheManager([PagedKV(1, 4)], 4, 8, 2, prefix_sharing=True).prefix is not None


# ------------------------------------------------------------------ the plain implementation, read a second time
def test_norm_and_embedding_element_by_element():
    g = torch.Generator().manual_seed(1)
    x, w = torch.randn(3, 5, generator=g, dtype=F64), torch.randn(5, generator=g, dtype=F64)
    got = plain.norm(x, w, 1e-3)
    for t in range(3):
        r = math.sqrt(sum(float(v) ** 2 for v in x[t]) / 5 + 1e-3)
        for i in range(5):
            assert abs(float(got[t, i]) - float(x[t, i]) / r * (1.0 + float(w[i]))) < 1e-12
    tables = {"embed": torch.randn(7, 4, generator=g, dtype=F64), "pos": torch.randn(9, 4, generator=g, dtype=F64)}
    assert torch.equal(plain.embedding(tables, [3, 6], start=5), torch.stack([tables["embed"][3] + tables["pos"][5],
                                                                            tables["embed"][6] + tables["pos"][6]]))


def test_what_is_visible():
    tokens, blocks = plain.visible(9, {"size": 4, "pool": 3})  # window 6..9; blocks 0..2 and 3..5 lie before it
    assert tokens == [6, 7, 8, 9] and blocks == [0, 1]
    tokens, blocks = plain.visible(8, {"size": 4, "pool": 3})  # window 5..8: block 1 holds 5; 3 and 4 are seen by nothing
    assert tokens == [5, 6, 7, 8] and blocks == [0]
    assert plain.visible(3, {"size": 4, "pool": 1}) == ([0, 1, 2, 3], [])
    assert plain.visible(4, {"size": 4, "pool": 1}) == ([1, 2, 3, 4], [0])
    assert plain.visible(5, {"size": 2}) == ([4, 5], []) and plain.visible(2, None) == ([0, 1, 2], [])
    for size, pool in ((5, 16), (1, 3), (24, 5), (16, 16)):
        for t in range(100):
            blocks = plain.visible(t, {"size": size, "pool": pool})[1]
            assert len(blocks) == max(0, t - size + 1) // pool  # what the kernels count by


def test_attention_by_hand():
    g = torch.Generator().manual_seed(5)
    W, H, G, d, dv, T, eps = 6, 4, 2, 3, 5, 11, 1e-4
    mixer = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": 0.8, "mask": {"size": 3, "pool": 2}, "v_mix": True}
    w = {"m.q": torch.randn(H * d, W, generator=g, dtype=F64), "m.k": torch.randn(G * d, W, generator=g, dtype=F64),
         "m.v": torch.randn(G * dv, W, generator=g, dtype=F64), "m.vmix": torch.tensor(0.3, dtype=F64),
         "m.q.norm": 1.0 + 0.1 * torch.randn(H * d, generator=g, dtype=F64),
         "m.k.norm": 1.0 + 0.1 * torch.randn(G * d, generator=g, dtype=F64), "m.o": torch.eye(H * dv, dtype=F64)}
    x, v1 = torch.randn(T, W, generator=g, dtype=F64), torch.randn(T, G * dv, generator=g, dtype=F64)
    got, _, own = plain.attention(x, w, "m", mixer, eps, first_values=v1)

    def project(name, t):
        return [sum(float(w[name][r, c]) * float(x[t, c]) for c in range(W)) for r in range(w[name].shape[0])]

    def normed(row, weight):
        r = math.sqrt(sum(a * a for a in row) / len(row) + eps)
        return [a / r * float(b) for a, b in zip(row, weight)]

    q = [normed(project("m.q", t), w["m.q.norm"]) for t in range(T)]
    k = [normed(project("m.k", t), w["m.k.norm"]) for t in range(T)]
    v = [[0.7 * a + 0.3 * float(b) for a, b in zip(project("m.v", t), v1[t])] for t in range(T)]
    assert all(abs(float(own[t, i]) - project("m.v", t)[i]) < 1e-12 for t in range(T) for i in range(G * dv))
    for t in range(T):
        keys = [(k[j], v[j]) for j in range(T) if 0 <= t - j < 3]
        for b in range(T):
            if 2 * b + 1 <= t - 3:
                keys.append(([(k[2 * b][i] + k[2 * b + 1][i]) / 2 for i in range(G * d)],
                             [(v[2 * b][i] + v[2 * b + 1][i]) / 2 for i in range(G * dv)]))
        for h in range(H):
            kv = h // 2
            s = [0.8 * sum(q[t][h * d + i] * kk[kv * d + i] for i in range(d)) for kk, _ in keys]
            den = sum(math.exp(z) for z in s)
            for c in range(dv):
                want = sum(math.exp(z) / den * vv[kv * dv + c] for z, (_, vv) in zip(s, keys))
                assert abs(float(got[t, h * dv + c]) - want) < 1e-10


def test_dense_by_hand():
    g = torch.Generator().manual_seed(6)
    W, ff, L = 4, 6, 0.8
    w = {"m.gate": 2.0 * torch.randn(ff, W, generator=g, dtype=F64), "m.up": 2.0 * torch.randn(ff, W, generator=g, dtype=F64),
         "m.down": torch.randn(W, ff, generator=g, dtype=F64)}
    x = torch.randn(5, W, generator=g, dtype=F64)
    got = plain.dense(x, w, "m", L)
    clipped = set()
    for t in range(5):
        a = []
        for j in range(ff):
            gt = sum(float(w["m.gate"][j, i]) * float(x[t, i]) for i in range(W))
            up = sum(float(w["m.up"][j, i]) * float(x[t, i]) for i in range(W))
            clipped |= {n for n, hit in (("gate", gt > L), ("low gate", gt < -L), ("up", up > L), ("low up", up < -L)) if hit}
            gt, up = min(gt, L), max(-L, min(L, up))
            a.append(gt / (1.0 + math.exp(-1.702 * gt)) * (up + 1.0))
        for c in range(W):
            assert abs(float(got[t, c]) - sum(float(w["m.down"][c, j]) * a[j] for j in range(ff))) < 1e-10
    assert clipped == {"gate", "low gate", "up", "low up"}  # the gate is cut from above only


def test_mixture_by_hand():
    g = torch.Generator().manual_seed(3)
    W, ff, E, top = 6, 4, 5, 2
    w = {"m.router": torch.randn(E, W, generator=g, dtype=F64)}
    for e in range(E):
        w[f"m.e{e}.gate"], w[f"m.e{e}.up"] = (torch.randn(ff, W, generator=g, dtype=F64) for _ in range(2))
        w[f"m.e{e}.down"] = torch.randn(W, ff, generator=g, dtype=F64)
    x = torch.randn(3, W, generator=g, dtype=F64)
    margins = [math.inf] * 3
    got = plain.mixture(x, w, "m", {"router": {"experts": E, "top": top}}, margins)
    for t in range(3):
        z = [sum(float(w["m.router"][e, i]) * float(x[t, i]) for i in range(W)) for e in range(E)]
        order = sorted(range(E), key=lambda e: -z[e])
        size = math.sqrt(sum(float(a) ** 2 for a in x[t]) / W) * math.sqrt(float((w["m.router"] ** 2).sum()) / E)
        assert abs(margins[t] - (z[order[1]] - z[order[2]]) / size) < 1e-12
        want = [0.0] * W
        for e in order[:top]:
            s = 1.0 / (1.0 + math.exp(-z[e]))
            a = []
            for j in range(ff):
                gt = sum(float(w[f"m.e{e}.gate"][j, i]) * s * float(x[t, i]) for i in range(W))
                up = sum(float(w[f"m.e{e}.up"][j, i]) * s * float(x[t, i]) for i in range(W))
                a.append(gt / (1.0 + math.exp(-gt)) * up)
            for c in range(W):
                want[c] += sum(float(w[f"m.e{e}.down"][c, j]) * a[j] for j in range(ff))
        assert all(abs(float(got[t, c]) - want[c]) < 1e-10 for c in range(W))


def test_values_are_mixed_with_the_first_mixing_layer_and_norms_stand_on_the_outputs():
    """One token, two layers of which both mix: the second one's output by hand."""
    cfg = cases.config([cases.layer(1, 1, 4, 4, (3, 2), None), cases.layer(1, 1, 4, 4, (3, 2), None)], width=4, vocab=5,
                       max_positions=4, eps=1e-5)
    w = {n: t.double() for n, t in cases.make_weights(cfg, 9).items()}
    seen = []
    plain.forward(cfg, w, [2], after_layer=lambda i, x: seen.append(x[0].clone()))
    x = w["embed"][2] + w["pos"][0]
    v1 = w["l0.mix.v"] @ x
    x = x + plain.norm(w["l0.mix.o"] @ v1, w["l0.norm1"], 1e-5)  # a token alone attends to itself
    assert torch.allclose(seen[0], x, atol=1e-12)
    lam = float(w["l1.mix.vmix"])
    v2 = (1.0 - lam) * (w["l1.mix.v"] @ x) + lam * v1
    x = x + plain.norm(w["l1.mix.o"] @ v2, w["l1.norm1"], 1e-5)
    assert torch.allclose(seen[1], x, atol=1e-12)


@pytest.mark.parametrize("case", sorted(cases.CASES))
def test_the_plain_implementation_cut_anywhere(case):
    """Whole, in portions, and token by token from an explicit state: the same logits."""
    cfg, weights = cases.CASES[case], cases.make_weights(cases.CASES[case], 7)
    ids = cases.random_ids(cfg["vocab"], 60, 3)
    whole, _ = plain.forward(cfg, weights, ids)
    rows, state, pos = [], None, 0
    for n in (1, 7, 2, 20, 1, 1, 28):
        logits, state = plain.forward(cfg, weights, ids[pos:pos + n], start=pos, state=state)
        rows.append(logits)
        pos += n
    assert float((torch.cat(rows) - whole).abs().max()) < 1e-9


def test_a_safe_sequence_has_no_close_call():
    cfg, weights = cases.CASE_A, cases.make_weights(cases.CASE_A, 7)
    ids, rows = cases.safe_sequence(cfg, weights, 30, 1)
    margins = [math.inf] * 30
    whole, _ = plain.forward(cfg, weights, ids, margins=margins)
    assert min(margins) >= cases.CLOSE_CALL * 0.999 and float((whole - rows).abs().max()) < 1e-9
