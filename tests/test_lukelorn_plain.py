"""The Lukelorn decoder without a GPU: its configuration and plan, what the cache manager does with a window that keeps the first
tokens, and a second reading of every function of the plain implementation, element by element with ``math`` alone."""

import copy
import math
import random

import pytest
import torch

import lukelorn_cases as cases
import plain_lukelorn as plain
from ferrisinfer_b200.cache.manager import NO_PAGE, CacheManager
from ferrisinfer_b200.config import resolve_config
from ferrisinfer_b200.errors import ConfigError, UnsupportedError, WeightLoadError
from ferrisinfer_b200.parts import build_model
from ferrisinfer_b200.parts.attention import GroupedQueryAttention
from ferrisinfer_b200.parts.base import CombinedNeed, FixedState, PagedKV
from ferrisinfer_b200.parts.block import ParallelResidualBlock, PreNormResidualBlock
from ferrisinfer_b200.parts.feed_forward import DenseActivation, MixtureOfExperts
from ferrisinfer_b200.parts.norm import GroupedRMSNorm
from ferrisinfer_b200.parts.plan import PartSpec
from ferrisinfer_b200.parts.position import ScaledRotary
from ferrisinfer_b200.weights.loader import check_tensors

F64 = torch.float64


# ------------------------------------------------------------------------------------------ configuration, plan
@pytest.mark.parametrize("case", sorted(cases.CASES))
def test_configuration_round_trip_and_tensor_names(case):
    cfg = cases.CASES[case]
    arch, c = resolve_config(copy.deepcopy(cfg))
    assert arch.name == "Lukelorn" and resolve_config(c.to_dict())[1] == c
    model = build_model(arch.plan(c))
    specs = model.tensor_specs()
    shapes = cases.tensor_shapes(cfg, cases.LOW_RANKS[case])
    assert {s.name for s in specs} == set(shapes) and all(s.required for s in specs)
    check_tensors(specs, shapes)
    with pytest.raises(WeightLoadError):
        check_tensors(specs, {n: s for n, s in shapes.items() if n != "l0.norm1"})
    assert len(model.plan.run_order) == len(cfg["layers"])


def test_layers_that_run_another_layers_tensors():
    """The tensors of a layer that runs again stand once; every run has a cache or state of its own."""
    arch, c = resolve_config(cases.CASES["B"])
    plan = arch.plan(c)
    assert [lp.prefix for lp in plan.layers] == ["l0", "l1", "l2", "l3"]
    assert [s.layer for s in plan.run_order] == [0, 1, 2, 3, 2, 3, 2, 1] and all(s.cache_of is None for s in plan.run_order)
    needs = build_model(plan).cache_needs()
    assert needs[0] == PagedKV(3, 24, 11, 20, keep_first=35) and needs[2] == needs[4] == needs[6] == PagedKV(1, 39, 30, 0)
    assert needs[7] == CombinedNeed((FixedState((2, 2 * 40 + 60)), FixedState((3, 20, 40))))
    mgr = CacheManager(needs, 16, 8, 2)
    assert [g.members for g in mgr.groups] == [[0], [2, 4, 6], [3, 5]]


def test_the_factor_on_what_layers_add_is_a_unit_of_the_residual_stream():
    arch, c = resolve_config(cases.CASES["C"])
    plan = arch.plan(c)
    assert plan.residual_unit == 1.7 and plan.embedding.params["scale"] == 1.0 / 1.7
    assert plan.final_norm.params["eps"] == plan.layers[0].mixer_norm.params["eps"] == pytest.approx(1e-5 / 1.7 ** 2)
    assert all(lp.feed_forward_norm is None for lp in plan.layers)
    # the norms inside mixers are of rows that carry no unit
    assert plan.layers[1].mixer.params["norm_eps"] == 1e-5
    x = torch.randn(3, 43, dtype=F64)
    assert torch.allclose(plain.rms_div(x, 1e-5), plain.rms_div(x / 1.7, 1e-5 / 1.7 ** 2), atol=1e-12)


def test_absent_keys():
    cfg = copy.deepcopy(cases.CASES["D"])
    del cfg["residual_mult"], cfg["layers"][4]
    for key in ("kv_heads", "vdim", "softcap", "rot", "mask"):
        del cfg["layers"][0]["mixer"][key]
    del cfg["layers"][1]["mixer"]["rot"]["dims"], cfg["layers"][1]["mixer"]["mask"], cfg["layers"][2]["mixer"]["kv_heads"]
    del cfg["layers"][3]["mixer"]["mask"]["keep_first"], cfg["layers"][3]["mixer"]["rot"]["scaling"], cfg["layers"][3]["mlp"]
    _, c = resolve_config(cfg)
    a, b, d, e = (x.mixer for x in c.layers)
    assert c.residual_mult == 1.0 and (a.kv_heads, a.vdim, a.softcap, a.rot.dims, a.window, a.keep_first) == (2, 128, None, 0, None, 0)
    assert b.rot.dims == 16 and b.window is None and d.kv_heads == 2
    assert e.keep_first == 0 and e.window == 16 and e.rot.scaling is None and c.layers[3].mlp is None


@pytest.mark.parametrize("change,error", [
    (lambda d: d["layers"][1]["mixer"].update(kv_heads=3), ConfigError),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=34), ConfigError),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=3), ConfigError),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("high"), ConfigError),
    (lambda d: d["layers"][1]["mixer"].update(softcap=-1.0), ConfigError),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(size=0), ConfigError),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(keep_first=-1), ConfigError),
    (lambda d: d["layers"][0]["mixer"].pop("q_rank"), ConfigError),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(keep_first=4), UnsupportedError),
    (lambda d: d["layers"][2]["mixer"].update(conv=0), ConfigError),
    (lambda d: d["layers"][1]["mlp"]["router"].update(top=7), ConfigError),
    (lambda d: d["layers"][1]["mlp"].update(kind="shared"), UnsupportedError),
    (lambda d: d["layers"][2].update(type="recurrent"), UnsupportedError),
    (lambda d: d["layers"][3].update(weights_of=9), ConfigError),
    (lambda d: d["layers"][3].update(weights_of=3), ConfigError),
    (lambda d: (d["layers"][3].update(weights_of=4), d["layers"][4].update(weights_of=3)), ConfigError),
    (lambda d: d["layers"][3].update(weights_of=2), ConfigError),  # another entry than that layer's
    (lambda d: d.update(residual_mult=0.0), ConfigError),
])
def test_configuration_errors(change, error):
    bad = copy.deepcopy(cases.CASES["A"])
    change(bad)
    with pytest.raises(error):
        resolve_config(bad)


def test_parts_refuse_what_does_not_go_together():
    base = dict(hidden_size=32, num_heads=2, num_kv_heads=1, head_dim=16, position=PartSpec("none"),
                tensor_names={n: n for n in "qkvo"})
    with pytest.raises(ValueError):  # first tokens are kept beside a window
        GroupedQueryAttention(keep_first=4, **base)
    with pytest.raises(ValueError):
        GroupedQueryAttention(window=8, keep_first=4, pool=2, qk_norm={"eps": 1e-6}, **base)
    with pytest.raises(ValueError):
        GroupedQueryAttention(softcap=-2.0, **base)
    with pytest.raises(ValueError):
        GroupedQueryAttention(output_gate={"name": "g", "kind": "silu", "per_head": True}, **base)
    with pytest.raises(ValueError):
        MixtureOfExperts(32, 16, 4, 2, gated=False, activation="gelu_tanh")
    with pytest.raises(ValueError):
        ScaledRotary(8, 1e4, scaling={"kind": "linear", "factor": 2.0})
    norm, ff = GroupedRMSNorm(32, 1e-6), DenseActivation(32, 16, "relu2")
    with pytest.raises(ValueError):  # one branch after the other: the second one needs a norm
        PreNormResidualBlock(32, GroupedQueryAttention(**base), ff, norm, None)
    ParallelResidualBlock(32, GroupedQueryAttention(**base), ff, norm, None)


@pytest.mark.parametrize("dims,base,scaling", [
    (32, 700.0, cases.SCALING), (16, 1e4, {"factor": 8.0, "low": 0.5, "high": 2.0, "original": 40.0}), (8, 50.0, None),
    (64, 5e5, {"factor": 16.0, "low": 2.0, "high": 3.0, "original": 4096.0})])
def test_frequencies(dims, base, scaling):
    """The table that the kernels take against the plain frequencies: 32-bit numbers and what they lack of 64-bit ones."""
    part = ScaledRotary(dims, base, "interleaved", None if scaling is None else {"kind": "wavelength", **scaling})
    table = part.table("cpu")
    want = plain.frequencies(dims, base, scaling)
    assert table.interleaved and table.magnitude == 1.0 and table.freq.dtype == torch.float32
    assert torch.allclose(table.freq.double(), want, rtol=1e-7, atol=0.0)
    assert torch.allclose(table.freq.double() + table.freq_lo.double(), want, rtol=1e-13, atol=0.0)
    if scaling is not None:  # every branch is there
        plainf = plain.frequencies(dims, base)
        ratio = want / plainf
        assert bool((ratio == 1.0).any()) and float(ratio.min()) == pytest.approx(1.0 / scaling["factor"])


# ------------------------------------------------------------------------------------------ the cache manager
@pytest.mark.parametrize("window,keep,page", [(24, 5, 16), (5, 35, 16), (1, 1, 4), (16, 16, 16), (16, 17, 8), (33, 0, 16), (7, 3, 1)])
def test_pages_of_a_window_that_keeps_the_first_tokens(window, keep, page):
    """Steps of changing size: every key that a token of the step reads has a page, and after the step no page is held that no
    later token can read."""
    mgr = CacheManager([PagedKV(2, 8, window, keep_first=keep)], page, 200 if page < 4 else 64, 2)
    mgr.admit("other"), mgr.extend("other", page + 1), mgr.commit("other", page + 1)
    mgr.admit("a")
    rng = random.Random(window * 1000 + keep * 10 + page)
    total, first_pages = 0, None
    while total < 3 * max(window, keep) + 60:
        n = rng.choice([1, 1, 2, 3, window // 2 + 1, window + 3])
        before, total = total, total + n
        mgr.extend("a", total)
        table = mgr.block_table("a", 0)
        for p in range(before, total):
            assert all(table[j // page] >= 0 for j in range(p + 1) if p - j < window or j < keep), p
        mgr.commit("a", total)
        table = mgr.block_table("a", 0)
        needed = {j // page for j in range(total) if total - j < window or j < keep}
        held = {b for b, x in enumerate(table) if x != NO_PAGE}
        assert needed <= held and held - needed <= {len(table) - 1, max(0, total - window + 1) // page}, (total, held, needed)
        kept = tuple(table[:min(-(-keep // page), total // page)])
        if first_pages is not None:
            assert kept[:len(first_pages)] == first_pages  # they never move
        first_pages = kept
        mgr.check_invariants()
    assert len(held) <= -(-keep // page) + -(-window // page) + 1
    mgr.release("a"), mgr.release("other")
    assert all(g.pool.num_used == 0 for g in mgr.groups)


def test_requests_that_keep_first_tokens_need_room_for_them():
    need = PagedKV(1, 4, 20, keep_first=30)
    assert need.span == 50 and need.first_needed(100) == 81 and not need.keeps_all
    assert CacheManager([need], 4, 8, 2, prefix_sharing=True).prefix is None


# ------------------------------------------------------------------ the plain implementation, read a second time
def rows(w, x):
    return [[sum(float(w[r, c]) * float(t[c]) for c in range(w.shape[1])) for r in range(w.shape[0])] for t in x]


def sigmoid(v):
    return 1.0 / (1.0 + math.exp(-v))


def turned(vec, p, freq):
    out = list(vec)
    for i, f in enumerate(freq):
        a, u, v = p * f, vec[2 * i], vec[2 * i + 1]
        out[2 * i], out[2 * i + 1] = u * math.cos(a) - v * math.sin(a), v * math.cos(a) + u * math.sin(a)
    return out


def drawn(shapes, seed):
    g = torch.Generator().manual_seed(seed)
    return {f"m.{n}": cases.draw(n, s, g).double() for n, s in shapes.items()}


def test_frequencies_by_hand():
    s = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 100.0}
    f = plain.frequencies(8, 1000.0, s)
    for i in range(4):
        raw = 1000.0 ** (-2.0 * i / 8)
        wave = 2.0 * math.pi / raw
        if wave < 25.0:
            want = raw
        elif wave > 100.0:
            want = raw / 4.0
        else:
            mix = (100.0 / wave - 1.0) / 3.0
            want = (1.0 - mix) * raw / 4.0 + mix * raw
        assert abs(float(f[i]) - want) < 1e-15
    assert float(f[0]) == 1.0 and float(f[3]) == pytest.approx(1000.0 ** -0.75 / 4.0)


def test_what_is_visible():
    ok = plain.seen(10, 10, size=3, keep_first=2)
    assert [j for j in range(10) if ok[9, j]] == [0, 1, 7, 8, 9]
    assert [j for j in range(10) if ok[3, j]] == [0, 1, 2, 3] and [j for j in range(10) if ok[0, j]] == [0]
    assert torch.equal(plain.seen(2, 10, size=3, keep_first=2), ok[8:])
    assert [j for j in range(6) if plain.seen(6, 6, size=1)[5, j]] == [5] and bool(plain.seen(6, 6)[5].all())


def test_attention_by_hand():
    W, T = 6, 9
    m = cases.attention(4, 2, 6, 5, (3, 2), None, rot=4, base=20.0, softcap=1.5, scale=0.8)["mixer"]
    w = drawn(cases.mixer_shapes("attention", m, W, None), 5)
    w["m.o"] = torch.eye(20, dtype=F64)
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(1), dtype=F64)
    got = plain.attention(x, w, "m", m, list(range(T)))[0]
    q, k, v, gate = (rows(w["m." + n], x) for n in ("q", "k", "v", "g"))
    freq = [float(f) for f in plain.frequencies(4, 20.0, cases.SCALING)]
    for t in range(T):
        for h in range(4):
            kv = h // 2
            qt = turned(q[t][6 * h:6 * h + 6], t, freq)
            keys = [j for j in range(t + 1) if t - j < 3 or j < 2]
            e = []
            for j in keys:
                s = 0.8 * sum(a * b for a, b in zip(qt, turned(k[j][6 * kv:6 * kv + 6], j, freq)))
                e.append(math.exp(1.5 * math.tanh(s / 1.5)))
            den = sum(e) + math.exp(float(w["m.sink"][h]))
            for c in range(5):
                want = sum(a / den * v[j][5 * kv + c] for a, j in zip(e, keys)) * sigmoid(gate[t][h])
                assert abs(float(got[t, 5 * h + c]) - want) < 1e-10


def test_latent_attention_by_hand():
    W, T, H, d, r, dv, qr, kr, eps = 6, 7, 2, 3, 2, 4, 5, 7, 1e-3
    m = cases.latent(H, d, r, dv, qr, kr, 4, None, base=9.0, scale=0.7)["mixer"]
    w = drawn(cases.mixer_shapes("latent_attention", m, W, None), 6)
    w["m.o"] = torch.eye(H * dv, dtype=F64)
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(2), dtype=F64)
    got = plain.latent_attention(x, w, "m", m, eps, list(range(T)))[0]

    def normed(row, weight):
        s = math.sqrt(sum(a * a for a in row) / len(row) + eps)
        return [a / s * float(b) for a, b in zip(row, weight)]

    dq, dkv, gate = (rows(w["m." + n], x) for n in ("dq", "dkv", "g"))
    q = rows(w["m.uq"], [torch.tensor(normed(c, w["m.dq.norm"]), dtype=F64) for c in dq])
    c = [torch.tensor(normed(a[:kr], w["m.dkv.norm"]), dtype=F64) for a in dkv]
    k, v = rows(w["m.uk"], c), rows(w["m.uv"], c)
    for t in range(T):
        for h in range(H):
            mine = q[t][h * (d + r):(h + 1) * (d + r)]
            keys = [j for j in range(T) if 0 <= t - j < 4]
            e = []
            for j in keys:
                s = sum(a * b for a, b in zip(mine[:d], k[j][h * d:(h + 1) * d]))
                s += sum(a * b for a, b in zip(turned(mine[d:], t, [1.0]), turned(dkv[j][kr:], j, [1.0])))
                e.append(math.exp(0.7 * s))
            for i in range(dv):
                want = sum(a / sum(e) * v[j][h * dv + i] for a, j in zip(e, keys)) * sigmoid(gate[t][h])
                assert abs(float(got[t, h * dv + i]) - want) < 1e-10


def test_channel_delta_by_hand():
    W, T, H, G, d, dv, taps, eps = 5, 6, 4, 2, 3, 2, 3, 1e-4
    m = cases.delta(H, G, d, dv, taps, None)["mixer"]
    w = drawn(cases.mixer_shapes("channel_delta", m, W, (2, 3)), 7)
    w["m.o"] = torch.eye(H * dv, dtype=F64)
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(3), dtype=F64)
    got = plain.channel_delta(x, w, "m", m, eps)[0]
    conv = {}
    for n in "qkv":
        raw, c = rows(w["m." + n], x), w[f"m.{n}.conv"]
        conv[n] = []
        for t in range(T):
            y = [sum(float(c[i, j]) * raw[t - taps + 1 + j][i] for j in range(taps) if t - taps + 1 + j >= 0) for i in range(len(raw[0]))]
            conv[n].append([a * sigmoid(a) for a in y])
    b = rows(w["m.b"], x)
    z = rows(w["m.a2"], [torch.tensor(a, dtype=F64) for a in rows(w["m.a1"], x)])
    gate = rows(w["m.g2"], [torch.tensor(a, dtype=F64) for a in rows(w["m.g1"], x)])
    for h in range(H):
        S = [[0.0] * dv for _ in range(d)]
        kh = h // 2
        for t in range(T):
            q, k = (conv[n][t][kh * d:(kh + 1) * d] for n in "qk")
            q = [a / math.sqrt(sum(y * y for y in q) + 1e-6) / math.sqrt(d) for a in q]
            k = [a / math.sqrt(sum(y * y for y in k) + 1e-6) for a in k]
            v = conv["v"][t][h * dv:(h + 1) * dv]
            for i in range(d):
                soft = math.log(1.0 + math.exp(z[t][h * d + i] + float(w["m.dt_bias"][h * d + i])))
                decay = math.exp(-math.exp(float(w["m.A_log"][h])) * soft)
                S[i] = [decay * s for s in S[i]]
            u = [sigmoid(b[t][h]) * (v[c] - sum(S[i][c] * k[i] for i in range(d))) for c in range(dv)]
            S = [[S[i][c] + k[i] * u[c] for c in range(dv)] for i in range(d)]
            o = [sum(S[i][c] * q[i] for i in range(d)) for c in range(dv)]
            r = math.sqrt(sum(a * a for a in o) / dv + eps)
            for c in range(dv):
                want = o[c] / r * float(w["m.norm"][c]) * sigmoid(gate[t][h * dv + c])
                assert abs(float(got[t, h * dv + c]) - want) < 1e-10


def test_feed_forwards_by_hand():
    W, ff, E, top = 5, 4, 6, 2
    shapes = {"gate": (ff, W), "up": (ff, W), "down": (W, ff), "router": (E, W)}
    for e in range(E):
        shapes[f"e{e}.up"], shapes[f"e{e}.down"] = (ff, W), (W, ff)
    w = drawn(shapes, 8)
    x = torch.randn(3, W, generator=torch.Generator().manual_seed(4), dtype=F64)
    got = plain.dense(x, w, "m")
    g, u = rows(w["m.gate"], x), rows(w["m.up"], x)
    for t in range(3):
        a = [p * sigmoid(p) * q for p, q in zip(g[t], u[t])]
        assert all(abs(float(got[t, c]) - sum(float(w["m.down"][c, j]) * a[j] for j in range(ff))) < 1e-10 for c in range(W))
    margins = [math.inf]
    got = plain.mixture(x, w, "m", {"router": {"experts": E, "top": top}}, margins)
    z = rows(w["m.router"], x)
    gaps = []
    for t in range(3):
        order = sorted(range(E), key=lambda e: -z[t][e])
        gaps.append(z[t][order[1]] - z[t][order[2]])
        want = [0.0] * W
        for e in order[:top]:
            up = [sum(float(w[f"m.e{e}.up"][j, i]) * sigmoid(z[t][e]) * float(x[t, i]) for i in range(W)) for j in range(ff)]
            for c in range(W):
                want[c] += sum(float(w[f"m.e{e}.down"][c, j]) * max(up[j], 0.0) ** 2 for j in range(ff))
        assert all(abs(float(got[t, c]) - want[c]) < 1e-10 for c in range(W))
    assert abs(margins[0] - min(gaps)) < 1e-12


def test_layers_add_both_branches_of_one_norm_with_a_factor():
    """One token, a layer that runs twice: by hand from the parts."""
    layer = cases.attention(1, 1, 4, 4, (3, 1), cases.dense(6))
    cfg = cases.config([layer, dict(layer, weights_of=0)], width=4, vocab=5, eps=1e-5, mult=0.7)
    w = {n: t.double() for n, t in cases.make_weights(cfg, 9).items()}
    assert not any(n.startswith("l1") for n in w)
    after = []
    logits, _ = plain.forward(cfg, w, [2], after=after)
    x = w["embed"][2]
    for i in range(2):
        h = x / math.sqrt(float((x * x).mean()) + 1e-5) * (1.0 + w["l0.norm1"])
        y = plain.attention(h[None], w, "l0.mix", layer["mixer"], [0])[0][0] + plain.dense(h[None], w, "l0.mlp")[0]
        x = x + 0.7 * y
        assert torch.allclose(after[i][0], x, atol=1e-12)
    assert torch.allclose(logits[0], w["head"] @ (x / math.sqrt(float((x * x).mean()) + 1e-5) * (1.0 + w["final.norm"])), atol=1e-12)


@pytest.mark.parametrize("case", sorted(cases.CASES))
def test_the_plain_implementation_cut_anywhere(case):
    """Whole, in portions, and token by token from an explicit state: the same logits."""
    cfg = cases.CASES[case]
    weights = {n: t.double() for n, t in cases.make_weights(cfg, 7, cases.LOW_RANKS[case]).items()}
    ids = cases.random_ids(cfg["vocab"], 60, 3)
    whole, _ = plain.forward(cfg, weights, ids)
    parts, state, pos = [], None, 0
    for n in (1, 7, 2, 20, 1, 1, 28):
        logits, state = plain.forward(cfg, weights, ids[pos:pos + n], start=pos, state=state)
        parts.append(logits)
        pos += n
    assert float((torch.cat(parts) - whole).abs().max()) < 1e-9


@pytest.mark.parametrize("case", ["A", "B"])
def test_every_mechanism_moves_the_logits(case):
    """What a fault of a mechanism would change is far above the tolerance of the comparisons on the GPU: a mechanism left out moves the logits of some position by more than the bfloat16 comparison lets pass (four tolerances); a window or the kept
    tokens off by one by a thousand times what the 32-bit comparison does (and, per kernel, loud keys show them in bfloat16)."""
    cfg = cases.CASES[case]
    weights = {n: t.double() for n, t in cases.make_weights(cfg, 7, cases.LOW_RANKS[case]).items()}
    ids = cases.random_ids(cfg["vocab"], 70, 3)
    want, _ = plain.forward(cfg, weights, ids)

    def moved(change_cfg=None, change_w=None):
        c, w = copy.deepcopy(cfg), dict(weights)
        if change_cfg:
            for e in c["layers"]:
                change_cfg(e["type"], e["mixer"])
        for n in w:
            if change_w:
                w[n] = change_w(n, w[n])
        return float(cases.row_errors(plain.forward(c, w, ids)[0], want).max())

    edge = 1000 * cases.TOLERANCE["float32"]
    far = 5 * cases.TOLERANCE["bfloat16"]
    windows = lambda by: lambda kind, m: m.get("mask", {}).update(size=m["mask"]["size"] + by) if m.get("mask") else None
    assert moved(windows(1)) > edge and moved(windows(-1)) > edge
    keeps = lambda by: lambda kind, m: m["mask"].update(keep_first=m["mask"]["keep_first"] + by) if kind == "attention" else None
    assert moved(keeps(1)) > edge and moved(keeps(-1)) > edge
    assert moved(lambda kind, m: m.pop("softcap", None)) > far
    assert moved(lambda kind, m: m.get("rot", {}).pop("scaling", None)) > far or case == "B"
    for name, change in (("sink", lambda t: t - 100.0), (".g", torch.zeros_like), ("A_log", lambda t: t - 30.0), (".g2", torch.zeros_like),
                         (".b", lambda t: t - 0.5), ("dt_bias", lambda t: t + 2.0), ("q.conv", lambda t: t.roll(1, -1))):
        assert moved(change_w=lambda n, t: change(t) if n.endswith(name) else t) > far, name


def test_a_safe_sequence_has_no_close_call():
    cfg, weights = cases.CASES["A"], cases.make_weights(cases.CASES["A"], 7, cases.LOW_RANKS["A"])
    ids, want = cases.safe_sequence(cfg, weights, 30, 1)
    margins = [math.inf]
    whole, _ = plain.forward(cfg, {n: t.double() for n, t in weights.items()}, ids, margins=margins)
    assert margins[0] >= cases.CLOSE_CALL and float((whole - want).abs().max()) < 1e-9
