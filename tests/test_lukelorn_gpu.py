"""The Lukelorn decoder on the GPU against the plain implementation (``plain_lukelorn``, float64): each kernel of its mechanisms
alone, every mixer as a part, then whole models of several small configurations driven through the step function the ways a
server drives it (whole prompts, token by token, portions down to two tokens, mixed batches over pages and slots that come
back), and greedy generation through the engine."""

import functools
import math
import random

import pytest
import torch

import helpers
import lukelorn_cases as cases
import plain_lukelorn as plain
from test_netinex_gpu import fake_ctx, paged, tol_of
from test_retezen_gpu import make_folder, make_runner, rounded

pytestmark = pytest.mark.gpu
F32, F64, BF16 = torch.float32, torch.float64, torch.bfloat16
DTYPES = {"float32": F32, "bfloat16": BF16}


def _ops():
    from ferrisinfer_b200.kernels import ops
    return ops


@functools.lru_cache(maxsize=None)
def weights_of(case: str):
    return cases.make_weights(cases.CASES[case], sum(map(ord, case)), cases.LOW_RANKS[case])


@functools.lru_cache(maxsize=None)
def wanted(case: str, n: int, seed: int):
    """(ids, float64 logits of every position) of a random sequence without a close call of any router."""
    return cases.safe_sequence(cases.CASES[case], weights_of(case), n, seed)


def check_rows(got: dict, want: dict, dtype: str, what: str):
    """``want``: request -> float64 logits of every position.  In bfloat16 a few positions amplify rounding several
    times over the typical error: at most one position in fifty may exceed the tolerance, none four times it."""
    worst, where, over, count = 0.0, None, 0, 0
    tol = cases.TOLERANCE[dtype]
    for rid, rows_want in want.items():
        n = rows_want.shape[0]
        rows = torch.stack([got[(rid, p)] for p in range(n)])
        assert torch.isfinite(rows).all(), f"{what}: request {rid} has logits that are not finite"
        err = cases.row_errors(rows, rows_want)
        over, count = over + int((err > tol).sum()), count + n
        if float(err.max()) > worst:
            worst, where = float(err.max()), (rid, int(err.argmax()))
    if dtype == "float32":
        assert worst <= tol, f"{what} ({dtype}): error {worst:.3g} at {where}"
    else:
        assert worst <= 4 * tol and over <= max(1, count // 50), \
            f"{what} ({dtype}): error {worst:.3g} at {where}, {over} of {count} positions over {tol}"


# =========================================================================================== attention kernels
def filled(device, dtype, keys, values, ps, seed):
    """Pages out of order that hold ``keys`` [T, nkv, d] and ``values`` [T, nkv, dv]: (k cache, v cache, block table)."""
    T, nkv, d = keys.shape
    blocks = -(-T // ps)
    order = torch.randperm(blocks + 2, generator=torch.Generator().manual_seed(seed))[:blocks]
    pad = blocks * ps - T

    def pages(x):
        x = torch.cat([x, x.new_zeros(pad, *x.shape[1:])]).view(blocks, ps, nkv, -1).transpose(1, 2)
        out = torch.full((blocks + 3, *x.shape[1:]), 50.0)  # rows that nobody may read
        out[order] = x.float()
        return out.to(dtype).to(device)
    return pages(keys), pages(values), order.int().view(1, -1).to(device)


def attend(ops, form, q, T, k, v, table, nh, nkv, d, dv, window, scale, keep, device, terms=None):
    """The last position's row of attention through one of the kernels' forms: portions, single tokens, single tokens whose keys
    are cut into shares; ``rows``: on tensor cores (bf16)."""
    from ferrisinfer_b200.engine.workspace import Workspace

    tiled = form.startswith("portion")
    last = T - 1
    ctx = fake_ctx(device, [T], [0], [0]) if tiled else fake_ctx(device, [1], [last], [0])
    rows = q if tiled else q[last:]
    out = torch.empty(rows.shape[0], nh * dv, device=device, dtype=q.dtype)
    extra = dict(max_kv_len=T, workspace=Workspace(device)) if "shares" in form else {}
    ops.set_attention_rows("rows" in form)
    try:
        ops.paged_attention_simt(rows.contiguous(), out, k, v, table, ctx.token_seq, ctx.positions, nh, nkv, d, window, scale,
                                 v_head_dim=dv, max_q_len=T if tiled else 1, keep_first=keep, score_slopes=terms, **extra)
    finally:
        ops.set_attention_rows(True)
    return out[-1].float().cpu().double().view(nh, dv)


FORMS = ["single", "portion", "shares", "single rows", "portion rows", "shares rows"]


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("nh,nkv,d,dv", [(4, 2, 32, 24), (8, 1, 64, 64), (3, 3, 15, 9), (4, 2, 128, 128)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_one_key_stands_out_at_each_edge(device, form, nh, nkv, d, dv, dtype):
    """One token's key is made loud in turn: the first and the last kept token, the token behind it, the token just before the
    window, the window's first and last.  What is seen takes nearly all the weight; what is not must leave the mean over
    everything visible.  Kept tokens inside the window, at its edge, far behind it, more of them than the window is long,
    their edge on and off a page's border."""
    ops = _ops()
    if "rows" in form and (dtype == F32 or not ops._lib().ferris_attention_rows_takes(nh, nkv, d, dv, 1)):
        pytest.skip("a geometry of the tensor-core forms in bfloat16")
    for window, keep, last in ((24, 5, 27), (24, 5, 28), (24, 5, 200), (5, 35, 39), (5, 35, 40), (5, 35, 300), (1, 1, 1), (1, 1, 50),
                               (16, 16, 47), (16, 16, 31), (16, 16, 32), (33, 17, 600), (19, 1, 64), (40, 3, 20), (64, 64, 255)):
        torch.manual_seed(window * 1000 + last)
        T = last + 1
        direction = torch.randn(d)
        direction /= direction.norm()
        seen = [j for j in range(T) if last - j < window or j < keep]
        values = torch.randn(T, nkv, dv)
        q = torch.zeros(T, nh * d)
        q[last] = (3.0 * direction).repeat(nh)
        of = torch.arange(nh) // (nh // nkv)
        for at in {0, keep - 1, keep, last - window, last - window + 1, last}:
            if not 0 <= at < T:
                continue
            keys = torch.zeros(T, nkv, d)
            keys[at] = 10.0 * direction
            k, v, table = filled(device, dtype, keys, values, 16, at)
            got = attend(ops, form, q.to(device, dtype), T, k, v, table, nh, nkv, d, dv, window, 1.0, keep, device)
            want = (values[at] if at in seen else values[seen].mean(0)).double()[of]  # exp(30) against exp(0) of the others
            tol = 1e-4 if dtype == F32 else 1.5e-2
            assert torch.allclose(got, want, atol=tol, rtol=tol), (window, keep, last, at, at in seen, got[0, :3], want[0, :3])


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("nh,nkv,d,dv", [(4, 2, 32, 24), (6, 2, 48, 40), (3, 3, 15, 9), (8, 2, 128, 128), (12, 1, 64, 64)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_soft_cap_sink_and_gates(device, form, nh, nkv, d, dv, dtype):
    """Scores far beyond the cap (its bend decides the weights), a sink that takes a fair share and is neither scaled nor capped,
    a gate per head; with a window that keeps tokens, with a window alone and with every key."""
    ops = _ops()
    if "rows" in form and (dtype == F32 or not ops._lib().ferris_attention_rows_takes(nh, nkv, d, dv, 1)):
        pytest.skip("a geometry of the tensor-core forms in bfloat16")
    T, of = 90, torch.arange(nh) // (nh // nkv)
    torch.manual_seed(nh * d)
    q, keys, values = torch.randn(T, nh * d).to(dtype), torch.randn(T, nkv, d).to(dtype), torch.randn(T, nkv, dv).to(dtype)
    sink, gates = 2.0 + torch.randn(nh), torch.randn(T, nh + 5).to(dtype)
    k, v, table = filled(device, dtype, keys, values, 16, 3)
    for window, keep, cap in ((20, 7, 3.0), (33, 0, 0.7), (0, 0, 2.0), (20, 7, 0.0)):
        scale = 3.0 / math.sqrt(d)
        s = torch.einsum("hd,shd->hs", q[-1].double().view(nh, d), keys.double()[:, of]) * scale
        if cap:
            assert float(s.abs().max()) > 2.0 * cap
        s = plain.capped(s, cap or None)
        want = plain.weighted_values(s[:, None], plain.seen(1, T, window or None, keep), values.double()[:, of], sink.double())[0]
        want = want * torch.sigmoid(gates[-1, 3:3 + nh].double())[:, None]
        gate = gates.to(device)[:, 3:3 + nh]
        terms = ops.ScoreTerms(sink=sink.to(device), softcap=cap, gate=gate if form.startswith("portion") else gate[-1:])
        got = attend(ops, form, q.to(device), T, k, v, table, nh, nkv, d, dv, window, scale, keep, device, terms)
        assert torch.allclose(got, want, **(dict(atol=2e-5, rtol=1e-4) if dtype == F32 else dict(atol=6e-3, rtol=1e-2))), (window, keep, cap)


@pytest.mark.parametrize("nh,nkv,d,dv", [(4, 2, 32, 24), (8, 1, 64, 40), (2, 2, 128, 128), (40, 2, 24, 8), (6, 3, 200, 136),
                                          (16, 4, 128, 128), (3, 3, 8, 256), (4, 4, 64, 64)])
@pytest.mark.parametrize("window,keep,cap", [(33, 7, 2.0), (100, 16, 0.0), (5, 40, 5.0), (0, 0, 1.0)])
def test_attention_on_tensor_cores_against_cuda_cores(device, nh, nkv, d, dv, window, keep, cap):
    """bf16 rows through the tensor-core forms and through the CUDA-core forms (fp32 throughout): the results differ by the last
    rounding only, in portions of several requests (one behind a cached prefix, one of a single token) and in single tokens,
    whole and in shares.  The values of neighbours nearly cancel, so that weights rounded to 16 bits would be far off."""
    ops = _ops()
    from ferrisinfer_b200.engine.workspace import Workspace

    torch.manual_seed(nh * d + window)
    ps, lengths, starts = 16, [150, 1, 70, 33], [0, 90, 41, 300]
    blocks = [-(-(a + b) // ps) for a, b in zip(lengths, starts)]
    order = torch.randperm(sum(blocks) + 3)
    tables = torch.full((len(lengths), max(blocks)), -1, dtype=torch.int32)
    at = 0
    for i, n in enumerate(blocks):
        tables[i, :n] = order[at:at + n].int()
        at += n
    kc = torch.randn(sum(blocks) + 3, nkv, ps, d).to(BF16).to(device)
    sign = torch.where(torch.arange(ps) % 2 == 0, 100.0, -100.0).view(1, 1, ps, 1)
    vc = (sign + torch.randn(sum(blocks) + 3, nkv, ps, dv)).to(BF16).to(device)
    sink = torch.randn(nh).to(device)
    for q_lens, first in ((lengths, starts), ([1] * 4, [a + b - 1 for a, b in zip(lengths, starts)])):
        ctx = fake_ctx(device, q_lens, first, [0] * 4)
        T = ctx.num_tokens
        q = torch.randn(T, nh * d + 8).to(BF16).to(device)[:, :nh * d]
        gate = torch.randn(T, nh).to(BF16).to(device)
        outs = []
        for on, extra in ((True, {}), (True, dict(max_kv_len=450, workspace=Workspace(device))), (False, {})):
            out = torch.full((T, nh * dv), 7.0, dtype=BF16, device=device)
            ops.set_attention_rows(on)
            try:
                ops.paged_attention_simt(q, out, kc, vc, tables.to(device), ctx.token_seq, ctx.positions, nh, nkv, d, window,
                                         1.5 / math.sqrt(d), score_slopes=ops.ScoreTerms(sink=sink, softcap=cap, gate=gate),
                                         v_head_dim=dv, max_q_len=max(q_lens), keep_first=keep, **extra)
            finally:
                ops.set_attention_rows(True)
            outs.append(out.float())
        for got in outs[:2]:
            err = (got - outs[2]).abs()
            assert bool((err <= 0.008 * outs[2].abs() + 3e-3).all()), (max(q_lens), float(err.max()))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("form", ["single", "portion", "shares", "single rows", "portion rows", "shares rows"])
@pytest.mark.parametrize("nh,rank,rot,window", [(4, 48, 8, 19), (3, 33, 6, 1), (2, 112, 16, 16), (16, 96, 32, 40), (20, 24, 8, 0),
                                                (2, 512, 64, 20)])
def test_latents_in_a_window_one_key_stands_out_at_each_edge(device, nh, rank, rot, window, form, dtype):
    """Keys that carry their values: the loud latent just inside the window takes the weight, the one just outside does not."""
    ops = _ops()
    from ferrisinfer_b200.engine.workspace import Workspace

    if "rows" in form and (dtype == F32 or rank % 8 or rot % 8):
        pytest.skip("a geometry of the tensor-core forms in bfloat16")
    row = rank + rot
    for last in (max(window - 1, 0), window, window + 1, 100, 300):
        T = last + 1
        seen = [j for j in range(T) if not window or last - j < window]
        torch.manual_seed(last)
        direction = torch.zeros(row)
        direction[rank:] = torch.randn(rot)  # the rotated part, which is no part of the value
        direction /= direction.norm()
        for at in {0, last - window, last - window + 1, last}:
            if not 0 <= at < T:
                continue
            latents = torch.zeros(T, 1, row)
            latents[:, 0, :rank] = torch.randn(T, rank)
            latents[at, 0, rank:] = 10.0 * direction[rank:]
            q = torch.zeros(T, nh * row)
            q[last] = (3.0 * direction).repeat(nh)
            k, _, table = filled(device, dtype, latents, latents, 16, at)
            portion = form.startswith("portion")
            ctx = fake_ctx(device, [T], [0], [0]) if portion else fake_ctx(device, [1], [last], [0])
            rows = q if portion else q[last:]
            out = torch.empty(rows.shape[0], nh * rank, device=device, dtype=dtype)
            extra = dict(max_kv_len=T, workspace=Workspace(device)) if "shares" in form else {}
            ops.set_attention_rows("rows" in form)
            try:
                ops.paged_attention_simt(rows.to(device, dtype), out, k, None, table, ctx.token_seq, ctx.positions, nh, 1, row, window, 1.0,
                                         v_head_dim=rank, max_q_len=T if portion else 1, values_in_keys=True, **extra)
            finally:
                ops.set_attention_rows(True)
            want = (latents[at, 0, :rank] if at in seen else latents[seen, 0, :rank].mean(0)).double()
            tol = 1e-4 if dtype == F32 else 1.5e-2
            assert torch.allclose(out[-1].cpu().double().view(nh, rank), want.expand(nh, rank), atol=tol, rtol=tol), (last, at)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_rotation_far_from_the_start(device, dtype):
    """Neighbours turned by scaled frequencies at positions up to 200,000: in 32-bit the angles keep more digits than one 32-bit
    product has."""
    ops = _ops()
    from ferrisinfer_b200.parts.position import ScaledRotary

    nh, nkv, d, dv, R = 3, 1, 24, 16, 16
    start, T = 199_990, 12
    rows = torch.randn(T, (nh + nkv) * d + nkv * dv).to(dtype)
    part = ScaledRotary(R, 5e4, "interleaved", {"kind": "wavelength", **cases.SCALING})
    ctx = fake_ctx(device, [T], [start], [0])
    k, _, _, slots = paged(device, dtype, T, nkv, d, 16, [1, 0])
    v = torch.zeros(*k.shape[:3], dv, dtype=dtype, device=device)
    x = rows.to(device)
    ops.qk_norm_rotary_cache_write(x, ctx, slots, k, v, nh, nkv, d, dv, None, None, 0.0, part.table(device))
    freq = plain.frequencies(R, 5e4, cases.SCALING)
    positions = list(range(start, start + T))
    want_q = plain.rotate_pairs(rows[:, :nh * d].double().view(T, nh, d), positions, freq)
    want_k = plain.rotate_pairs(rows[:, nh * d:(nh + nkv) * d].double().view(T, nkv, d), positions, freq)
    tol = dict(atol=2e-6, rtol=2e-6) if dtype == F32 else dict(atol=1e-3, rtol=8e-3)
    assert torch.allclose(x[:, :nh * d].cpu().double().view(T, nh, d), want_q, **tol)
    flat = lambda t: t.cpu().double().permute(0, 2, 1, 3).reshape(-1, t.shape[1], t.shape[-1])[slots.cpu().long()]
    assert torch.allclose(flat(k), want_k, **tol)
    assert torch.equal(flat(v), rows[:, (nh + nkv) * d:].double().view(T, nkv, dv))


# =========================================================================================== recurrence
def delta_inputs(T, heads, qk_heads, dim, vdim, seed, lo=-6.0):
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(*s, generator=g)
    z = lo + 6.0 * torch.rand(T, heads * dim, generator=g)
    return (rn(T, qk_heads * dim), rn(T, qk_heads * dim) / math.sqrt(dim), rn(T, heads * vdim), z, torch.rand(T, heads, generator=g))


def plain_delta(q, k, v, z, beta, rates, heads, qk_heads, dim, vdim):
    of = torch.arange(heads) // (heads // qk_heads)
    T = q.shape[0]
    g = torch.exp(-rates.double()[None, :, None] * plain.softplus(z.double()).view(T, heads, dim))
    return plain.channel_delta_scan(q.double().view(T, qk_heads, dim)[:, of], k.double().view(T, qk_heads, dim)[:, of],
                                    v.double().view(T, heads, vdim), g, beta.double(), torch.zeros(heads, dim, vdim, dtype=F64))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,qk_heads,dim,vdim", [(4, 2, 32, 24), (3, 3, 15, 9), (2, 1, 64, 64), (6, 2, 100, 33), (2, 2, 128, 128),
                                                      (1, 1, 256, 40), (3, 1, 8, 5)])
def test_delta_rule_with_a_decay_per_channel(device, heads, qk_heads, dim, vdim, dtype):
    """Whole, in portions and token by token, from a slot between others; the form that walks the tokens, the one that takes
    sixteen at a time (portions of no multiple of sixteen too), and whichever a step would take."""
    ops = _ops()
    T = 150
    q, k, v, z, beta = delta_inputs(T, heads, qk_heads, dim, vdim, heads * dim)
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    rates = torch.rand(heads) + 0.3
    want, last = plain_delta(q, k, v, z, beta, rates, heads, qk_heads, dim, vdim)
    want = want.reshape(T, heads * vdim)
    dev = lambda t: t.to(device)
    for cuts, chunks in (([T], None), ([70, 1, 50, 2, 27], None), ([100] + [1] * 50, None), ([2] * 20 + [64, 46], None),
                         ([T], False), ([T], True), ([16, 48, 17, 1, 2, 15, 33, 18], True), ([1] * 20 + [130], True)):
        state = torch.randn(3, heads, vdim, dim, device=device)
        others = state[:2].clone()
        state[2] = 0.0
        pos = 0
        for n in cuts:
            ctx = fake_ctx(device, [n], [pos], [2])
            sl = slice(pos, pos + n)
            out = torch.empty(n, heads * vdim, device=device)
            ops.gated_recurrence(dev(q[sl]), dev(k[sl]), dev(v[sl]), None, dev(beta[sl]), out, state, ctx, heads, qk_heads, dim, vdim,
                                 delta_rule=True, row_decay=(dev(z[sl]), dev(rates)), chunks=chunks)
            assert torch.allclose(out.cpu().double(), want[sl], atol=1e-4, rtol=2e-4), (cuts[:3], chunks, pos)
            pos += n
        assert torch.allclose(state[2].cpu().double().transpose(1, 2), last, atol=1e-4, rtol=2e-4)  # S lies transposed
        assert torch.equal(state[:2], others)


def test_delta_rule_of_several_requests_keeps_their_states_apart(device):
    """A long portion, two single tokens and a short one in one step, over slots out of order; later steps continue some of them;
    a write that is switched off leaves the states as they were."""
    ops = _ops()
    heads, qk_heads, dim, vdim = 4, 2, 32, 48
    lens = [130, 12, 9, 250]
    rates = torch.tensor([0.5, 1.0, 0.2, 2.0])
    data = [delta_inputs(n, heads, qk_heads, dim, vdim, n) for n in lens]
    want = [plain_delta(*d, rates, heads, qk_heads, dim, vdim)[0].reshape(n, heads * vdim) for d, n in zip(data, lens)]
    state = torch.zeros(6, heads, vdim, dim, device=device)
    slots, done = [4, 1, 5, 0], [0, 0, 0, 0]
    for step in ([100, 1, 1, 33], [30, 1, 0, 217], [0, 10, 8, 0]):
        live = [i for i in range(4) if step[i]]
        ctx = fake_ctx(device, [step[i] for i in live], [done[i] for i in live], [slots[i] for i in live])
        cat = lambda j: torch.cat([data[i][j][done[i]:done[i] + step[i]] for i in live]).to(device)
        out = torch.empty(sum(step), heads * vdim, device=device)
        before = state.clone()
        for write in (False, True):
            assert torch.equal(state, before)
            ops.gated_recurrence(cat(0), cat(1), cat(2), None, cat(4), out, state, ctx, heads, qk_heads, dim, vdim, delta_rule=True,
                                 row_decay=(cat(3), rates.to(device)), write_state=write)
        at = 0
        for i in live:
            assert torch.allclose(out[at:at + step[i]].cpu().double(), want[i][done[i]:done[i] + step[i]], atol=1e-4, rtol=2e-4)
            at += step[i]
            done[i] += step[i]
    assert done == lens


def test_delta_rule_whose_channels_forget_at_once(device):
    """Decays of e^-40 a token beside decays of almost one in the same head: nothing overflows, nothing is lost."""
    ops = _ops()
    heads, dim, vdim, T = 2, 32, 16, 100
    q, k, v, z, beta = delta_inputs(T, heads, heads, dim, vdim, 3)
    z = torch.where(torch.arange(heads * dim) % 3 == 0, torch.full_like(z, 40.0), torch.where(torch.rand_like(z) < 0.2, z + 30.0, z))
    rates = torch.ones(heads)
    want = plain_delta(q, k, v, z, beta, rates, heads, heads, dim, vdim)[0].reshape(T, -1)
    dev = lambda t: t.to(device)
    for chunks in (False, True):
        state, out = torch.zeros(1, heads, vdim, dim, device=device), torch.empty(T, heads * vdim, device=device)
        ops.gated_recurrence(dev(q), dev(k), dev(v), None, dev(beta), out, state, fake_ctx(device, [T], [0], [0]), heads, heads, dim, vdim,
                             delta_rule=True, row_decay=(dev(z), dev(rates)), chunks=chunks)
        assert torch.allclose(out.cpu().double(), want, atol=1e-4, rtol=2e-4), chunks


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_a_channel_that_hardly_forgets_over_thousands_of_tokens(device, dtype):
    """What token 3 wrote along one channel is read 3,000 tokens later: that channel's decay is within 1e-5 of one (a rounding of
    it to 24 bits at every step would show), the other channels forget fast."""
    ops = _ops()
    dim, vdim, T = 64, 32, 3000
    torch.manual_seed(5)
    k = torch.zeros(T, dim)
    k[:, 1:] = torch.randn(T, dim - 1) / math.sqrt(dim)
    k[3] = 0.0
    k[3, 0] = 1.0  # the only key along the first channel
    v, q = torch.randn(T, vdim), torch.zeros(T, dim)
    q[:, 0] = 1.0
    k, q, v = k.to(dtype), q.to(dtype), v.to(dtype)
    z = torch.full((T, dim), 1.0)
    z[:, 0] = -12.0 + torch.rand(T)
    rates, beta = torch.tensor([0.7]), torch.ones(T, 1)
    logs = -0.7 * plain.softplus(z[4:, 0].double()).sum()
    state = torch.zeros(1, 1, vdim, dim, device=device)
    pos, got = 0, None
    dev = lambda t: t.to(device)
    for n in [1000, 1, 900, 999, 60] + [1] * 40:
        ctx = fake_ctx(device, [n], [pos], [0])
        sl = slice(pos, pos + n)
        got = torch.empty(n, vdim, device=device)
        ops.gated_recurrence(dev(q[sl]), dev(k[sl]), dev(v[sl]), None, dev(beta[sl]), got, state, ctx, 1, 1, dim, vdim, delta_rule=True,
                             row_decay=(dev(z[sl]), dev(rates)))
        pos += n
    want = torch.exp(logs) * v[3].double()
    assert float((got[-1].cpu().double() - want).abs().max()) < 2e-5 * float(want.abs().max())


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("channels,taps", [(48, 4), (130, 2), (64, 3), (33, 4), (40, 1), (24, 5)])
def test_convolution_of_unequal_requests_in_one_step(device, channels, taps, dtype):
    """Portions, single tokens and long prompts side by side over slots out of order, continued in later steps; runs of tokens that
    begin and end inside requests; a slice of wider rows."""
    ops = _ops()
    torch.manual_seed(channels * taps)
    lens = [70, 1, 40, 3, 19]
    w = torch.randn(channels, taps)
    xs = [torch.randn(n + 30, channels).to(dtype) for n in lens]
    want = [plain.silu(plain.causal_conv(x.double(), w.double())[0]) for x in xs]
    state = torch.zeros(7, taps - 1, channels, device=device) if taps > 1 else None
    slots, done = [3, 0, 5, 1, 6], [0] * 5
    for step in (lens, [1] * 5, [2, 17, 1, 25, 11], [27, 12, 28, 4, 18]):
        live = [i for i in range(5) if step[i]]
        ctx = fake_ctx(device, [step[i] for i in live], [done[i] for i in live], [slots[i] for i in live])
        rows = torch.cat([xs[i][done[i]:done[i] + step[i]] for i in live])
        wide = torch.randn(rows.shape[0], channels + 10).to(dtype).to(device)
        wide[:, :channels] = rows.to(device)
        out = torch.empty(rows.shape[0], channels, dtype=dtype, device=device)
        ops.short_conv(wide[:, :channels], out, w.to(device), state, ctx, residual=False, silu=True)
        at = 0
        for i in live:
            assert torch.allclose(out[at:at + step[i]].cpu().double(), want[i][done[i]:done[i] + step[i]], **tol_of(dtype)), (step, i)
            at, done[i] = at + step[i], done[i] + step[i]
    assert done == [n + 30 for n in lens]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T", [1, 47, 48, 200])
@pytest.mark.parametrize("heads,K,N,pad", [(3, 64, 128, 16), (4, 48, 40, 8), (2, 200, 72, 0), (5, 13, 21, 3), (16, 128, 192, 64)])
def test_product_per_head(device, T, heads, K, N, pad, dtype):
    """Heads apart by more than their sizes, gates, sizes of whole tiles and not; short steps and those on tensor cores."""
    ops = _ops()
    torch.manual_seed(T + K)
    x, w = torch.randn(T, heads * (K + pad)).to(dtype), (torch.randn(heads, K, N) / math.sqrt(K)).to(dtype)
    gates = torch.randn(T, heads + 2).to(dtype)
    out = torch.full((T, heads * (N + 8)), 9.0, dtype=dtype, device=device)
    want = torch.einsum("thk,hkn->thn", x.double().view(T, heads, K + pad)[..., :K], w.double())
    ops.head_gemm(x.to(device), K + pad, w.to(device), out, N + 8)
    got = out.view(T, heads, N + 8)
    assert torch.allclose(got[..., :N].cpu().double(), want, **tol_of(dtype)) and bool((got[..., N:] == 9.0).all())
    ops.head_gemm(x.to(device), K + pad, w.to(device), out, N + 8, gate=gates.to(device)[:, 1:1 + heads])
    want = want * torch.sigmoid(gates[:, 1:1 + heads].double())[..., None]
    assert torch.allclose(out.view(T, heads, N + 8)[..., :N].cpu().double(), want, **tol_of(dtype))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,dv", [(3, 64), (2, 128), (4, 33), (1, 512), (2, 700), (5, 8), (2, 200)])
@pytest.mark.parametrize("kind", ["sigmoid", "silu"])
def test_norm_per_head_with_its_gate(device, heads, dv, kind, dtype):
    ops = _ops()
    torch.manual_seed(heads * dv)
    T = 37
    o, w, gate = 2.0 * torch.randn(T, heads * dv), 1.0 + 0.2 * torch.randn(dv), torch.randn(T, heads * dv + 8).to(dtype)
    g = gate[:, :heads * dv].double()
    want = (plain.rms_div(o.double().view(T, heads, dv), 1e-4) * w.double()).reshape(T, -1) * (torch.sigmoid(g) if kind == "sigmoid" else plain.silu(g))
    out = torch.empty(T, heads * dv, dtype=dtype, device=device)
    ops.gated_group_norm(o.to(device), gate.to(device)[:, :heads * dv], w.to(device), 1e-4, out, group=dv, gate_kind=kind)
    assert torch.allclose(out.cpu().double(), want, **tol_of(dtype))
    ops.gated_group_norm(o.to(device), None, w.to(device), 1e-4, out, group=dv)
    assert torch.allclose(out.cpu().double(), (plain.rms_div(o.double().view(T, heads, dv), 1e-4) * w.double()).reshape(T, -1), **tol_of(dtype))


# =========================================================================================== experts
@pytest.mark.parametrize("dtype,form", [(F32, "few"), (BF16, "few"), (BF16, "sorted"), (F32, "token"), (BF16, "token")])
@pytest.mark.parametrize("activation", ["relu2", "silu"])
@pytest.mark.parametrize("T,W,ff,E,top", [(1, 40, 24, 5, 1), (9, 44, 36, 12, 3), (70, 64, 96, 3, 3), (300, 128, 64, 8, 2),
                                           (17, 43, 33, 6, 4), (700, 256, 384, 16, 1)])
def test_experts_without_a_gate(device, T, W, ff, E, top, activation, dtype, form):
    """Router and experts together through the part in every form (an expert's weights read once for its tokens, a block per
    token, sorted by expert on tensor cores), replacing the rows and adding into them."""
    ops = _ops()
    from ferrisinfer_b200.parts.feed_forward import MixtureOfExperts

    if form == "sorted" and (W % 8 or ff % 8):
        pytest.skip("rows of no multiple of 8 elements are not sorted")
    torch.manual_seed(T + W)
    w = {"m.router": 1.5 * torch.randn(E, W) / math.sqrt(W)}
    for e in range(E):
        w[f"m.e{e}.up"], w[f"m.e{e}.down"] = 1.5 * torch.randn(ff, W) / math.sqrt(W), torch.randn(W, ff) / math.sqrt(ff)
    w = rounded(w)
    y = torch.randn(T, W).to(dtype)
    w64 = {n: t.double() for n, t in w.items()}
    chosen, weights, margin = plain.router(y.double(), w64, "m", top)
    want = torch.zeros(T, W, dtype=F64)
    act = (lambda a: torch.clamp(a, min=0.0) ** 2) if activation == "relu2" else plain.silu
    for t in range(T):
        for e, s in zip(chosen[t].tolist(), weights[t]):
            want[t] += act(s * y[t].double() @ w64[f"m.e{e}.up"].T) @ w64[f"m.e{e}.down"].T
    if activation == "relu2" and T < 100:
        assert torch.allclose(want, plain.mixture(y.double(), w64, "m", {"router": {"experts": E, "top": top}}), atol=1e-12)
    part = MixtureOfExperts(W, ff, E, top, router_bias_name=None, sigmoid_scores=True, input_weights=True, gated=False,
                            activation=activation)
    assert {s.name for s in part.tensor_specs("m")} == set(w)
    part.bind({n: t.to(device, dtype) for n, t in w.items()}, "m")
    was = ops.MOE_GROUPED_MIN_TOKENS, ops.MOE_FEW_MAX_PAIRS
    ops.MOE_GROUPED_MIN_TOKENS = 1 if form == "sorted" else 1 << 30
    ops.MOE_FEW_MAX_PAIRS = 0 if form == "token" else was[1]
    try:
        h = torch.full((T, W), 7.0, device=device)
        ctx = fake_ctx(device, [T], [0], [0], act_dtype=dtype)
        part.forward(y.to(device), h, ctx, accumulate=False)
        sure = margin > 1e-3  # a choice that a rounding of the sums could turn is not compared
        assert sure.sum() >= T * 0.8
        assert torch.allclose(h.cpu().double()[sure], want[sure], **tol_of(dtype, 3.0))
        part.forward(y.to(device), h, ctx)
        assert torch.allclose(h.cpu().double()[sure], 2.0 * want[sure], **tol_of(dtype, 6.0))
    finally:
        ops.MOE_GROUPED_MIN_TOKENS, ops.MOE_FEW_MAX_PAIRS = was


# =========================================================================================== mixers as parts
def mixers():
    """(name, type, mixer entry, inner sizes) of every mixer of the cases."""
    out = []
    for case, cfg in sorted(cases.CASES.items()):
        out += [pytest.param(e["type"], e["mixer"], cfg["norm"]["eps"], cases.LOW_RANKS[case], id=f"{case}{i}-{e['type']}")
                for i, e in enumerate(cfg["layers"]) if e.get("weights_of") is None]
    return out


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("kind,m,eps,ranks", mixers())
def test_mixer_against_the_plain_mixer(device, kind, m, eps, ranks, dtype):
    """Every mixer as a part (products, norms, rotation, cache or state, attention or recurrence, gate, output product): whole, as
    portions behind a cached prefix, and token by token, over pages out of order, against the plain mixer."""
    from ferrisinfer_b200.cache.manager import CacheManager
    from ferrisinfer_b200.config.lukelorn import _MIXERS
    from ferrisinfer_b200.models.lukelorn import _mixer
    from ferrisinfer_b200.parts.base import PagedMeta
    from ferrisinfer_b200.parts.plan import build_part

    W, T, ps = 48, 90, 16
    g = torch.Generator().manual_seed(len(str(m)))
    w = rounded({f"m.{n}": cases.draw(n, s, g) for n, s in cases.mixer_shapes(kind, m, W, ranks).items()})
    y = torch.randn(T, W, generator=g).to(dtype)
    w64 = {n: t.double() for n, t in w.items()}
    if kind == "attention":
        want = plain.attention(y.double(), w64, "m", m, list(range(T)))[0]
    elif kind == "latent_attention":
        want = plain.latent_attention(y.double(), w64, "m", m, eps, list(range(T)))[0]
    else:
        want = plain.channel_delta(y.double(), w64, "m", m, eps)[0]
    part = build_part("mixer", _mixer(kind, _MIXERS[kind].read(m, "here"), W, eps))
    roles = {s.name: s.role for s in part.tensor_specs("m")}
    assert set(roles) == set(w)
    part.bind({n: t.to(device, dtype if roles[n] == "matrix" else F32) for n, t in w.items()}, "m")
    for cuts in ([T], [40, 17] + [1] * 33, [2] * 30 + [1] * 30, [50] + [1] * 40):
        mgr = CacheManager([part.cache_need()], ps, 12, 2, dtype=dtype, device=device)
        mgr.admit("other"), mgr.extend("other", 20), mgr.commit("other", 20)
        mgr.admit("a")
        pos = 0
        for n in cuts:
            mgr.extend("a", pos + n)
            ctx = fake_ctx(device, [n], [pos], [mgr.get("a").slot], act_dtype=dtype)
            for grp in mgr.groups:
                ctx.paged[grp.gid] = PagedMeta(torch.tensor([mgr.block_table("a", grp.gid)], dtype=torch.int32, device=device),
                                               torch.tensor(mgr.slots_for("a", grp.gid, pos, n), dtype=torch.int32, device=device), ps)
            h = torch.ones(n, W, device=device)
            part.forward(y[pos:pos + n].to(device).contiguous(), h, ctx, mgr.layer_caches[0], True)
            # (32-bit: the delta rule divides a head's few values by their own size, which may be small)
            tol = tol_of(dtype, 5.0)
            assert torch.allclose(h.cpu().double() - 1.0, want[pos:pos + n], **tol), (cuts[:2], pos)
            mgr.commit("a", pos + n)
            pos += n


# ================================================================================================ whole models
MODEL_CASES = sorted(cases.CASES)
LENGTHS = {"long": (150, 11), "mid": (67, 12), "short": (23, 13), "one": (1, 14), "edge": (49, 15)}


def requests_of(case, names, lengths=LENGTHS):
    return {n: wanted(case, *lengths[n])[0] for n in names}


def rows_of(case, names, lengths=LENGTHS):
    return {n: wanted(case, *lengths[n])[1] for n in names}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", MODEL_CASES)
def test_whole_prompts(device, case, dtype):
    """Also the first tokens of a sequence: every position's logits are compared, from position 0 on."""
    runner = make_runner(cases.CASES[case], weights_of(case), dtype, device)
    names = ["long", "one", "short", "edge"]
    got = helpers.replay(runner, helpers.trace_whole(requests_of(case, names)))
    check_rows(got, rows_of(case, names), dtype, f"whole prompts {case}")
    runner.cache.check_invariants()
    assert runner.cache.num_free_slots == 4 and all(g.pool.num_used == 0 for g in runner.cache.groups)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", MODEL_CASES)
def test_every_layer_against_the_plain_layers(device, case, dtype):
    """The residual stream after every layer in the model's own units, not only the logits."""
    runner = make_runner(cases.CASES[case], weights_of(case), dtype, device, graphs=False)
    ids = wanted(case, *LENGTHS["edge"])[0]
    want = []
    plain.forward(cases.CASES[case], {n: t.double() for n, t in weights_of(case).items()}, ids, after=want)
    got = []
    runner.model.after_run = lambda i, h: got.append(h.detach().clone().cpu())
    helpers.replay(runner, helpers.trace_whole({"a": ids}))
    assert len(got) == len(want)
    for i, (g, w) in enumerate(zip(got, want)):
        scale = float(w.abs().max())
        assert float((g.double() - w).abs().max()) <= (1e-4 if dtype == "float32" else 6e-2) * scale, (case, i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", MODEL_CASES)
def test_token_by_token_from_the_first_token(device, case, dtype):
    """A long decode: 150 single tokens through recorded steps, over page borders and windows."""
    runner = make_runner(cases.CASES[case], weights_of(case), dtype, device)
    got = helpers.replay(runner, helpers.trace_tail_decoded(requests_of(case, ["long"]), tail=149))
    check_rows(got, rows_of(case, ["long"]), dtype, f"token by token {case}")
    assert runner.graph_replays > 100  # the decode steps were replayed from graphs


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", MODEL_CASES)
def test_prompt_then_decoded_tail(device, case, dtype):
    runner = make_runner(cases.CASES[case], weights_of(case), dtype, device, graphs=False)
    names = ["long", "mid", "edge"]
    got = helpers.replay(runner, helpers.trace_tail_decoded(requests_of(case, names), tail=40))
    check_rows(got, rows_of(case, names), dtype, f"prompt then single tokens {case}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", MODEL_CASES)
@pytest.mark.parametrize("sizes", [(2,), (7, 2, 13, 3, 5, 2, 16, 4, 9, 2, 31, 6), (64, 1, 2, 17)])
def test_portions(device, case, dtype, sizes):
    runner = make_runner(cases.CASES[case], weights_of(case), dtype, device)
    names = ["long", "short"] if sizes != (2,) else ["mid"]
    got = helpers.replay(runner, helpers.trace_portions(requests_of(case, names), sizes=sizes))
    check_rows(got, rows_of(case, names), dtype, f"portions of {sizes} {case}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", MODEL_CASES)
def test_mixed_batches_over_few_pages_and_slots(device, case, dtype):
    """Seven requests, at most three live, in a pool of three state slots and just enough pages: portions of some beside
    single tokens of others, requests that sit a step out, slots and pages that are used again by the next request."""
    names = ["mid", "short", "long", "one", "edge", "mid2", "short2"]
    lengths = dict(LENGTHS, mid2=(80, 21), short2=(30, 22))
    reqs = requests_of(case, names, lengths)
    steps = helpers.trace_mixed(reqs, seed=5, max_live=3)
    pages = helpers.tokens_held(steps, round_to=16) // 16
    runner = make_runner(cases.CASES[case], weights_of(case), dtype, device, num_pages=pages, max_requests=3)
    got = helpers.replay(runner, steps)
    check_rows(got, rows_of(case, names, lengths), dtype, f"mixed batches {case}")
    runner.cache.check_invariants()
    assert runner.cache.num_free_slots == 3 and all(g.pool.num_used == 0 for g in runner.cache.groups)


@pytest.mark.parametrize("case", ["A", "C"])
def test_a_batch_gives_every_request_what_it_gets_alone(device, case):
    """Unequal requests in one step, whole and then decoding together, against each of them alone."""
    names = ["long", "one", "short", "edge"]
    reqs = requests_of(case, names)
    alone = helpers.replay(make_runner(cases.CASES[case], weights_of(case), "float32", device), helpers.trace_whole(reqs))
    entries = [{"id": n, "tokens": ids[:max(1, len(ids) - 9)], "want": list(range(max(1, len(ids) - 9)))} for n, ids in reqs.items()]
    steps = [{"step": 0, "entries": entries, "end": ["one"]}]
    for i in range(9):
        steps.append({"step": i + 1, "end": [], "entries": [
            {"id": n, "tokens": [reqs[n][len(reqs[n]) - 9 + i]], "want": [0]} for n in names if n != "one"]})
    together = helpers.replay(make_runner(cases.CASES[case], weights_of(case), "float32", device), steps)
    for key, row in alone.items():
        assert torch.allclose(together[key], row, atol=4e-5, rtol=4e-5), key


def test_pages_behind_the_window_come_back_and_the_first_tokens_stay(device):
    """A pool far smaller than the request: the pages behind the window carry it on, the kept tokens' pages stay."""
    case = "A"  # windows of 19 and 24, five kept tokens
    ids, want = wanted(case, *LENGTHS["long"])
    runner = make_runner(cases.CASES[case], weights_of(case), "float32", device, num_pages=6, max_requests=1)
    got = helpers.replay(runner, helpers.trace_portions({"a": ids}, sizes=(9, 1, 2, 30, 1, 1, 5)))
    check_rows(got, {"a": want}, "float32", "few pages")
    assert all(g.pool.num_used == 0 for g in runner.cache.groups)


def test_pages_and_slots_used_again_by_the_next_request(device):
    """One slot and just enough pages: the second request takes what the first one left (keys, latents, states, convolutions), and
    computes what it computes alone."""
    case = "B"
    runner = make_runner(cases.CASES[case], weights_of(case), "float32", device, num_pages=10, max_requests=1)
    names = ["long", "mid"]
    got = helpers.replay(runner, helpers.trace_portions(requests_of(case, names), sizes=(40, 3, 1)))
    check_rows(got, rows_of(case, names), "float32", "pages used again")


@pytest.mark.parametrize("case,dtype", [("A", "float32"), ("A", "bfloat16"), ("B", "float32"), ("C", "float32")])
def test_a_long_prompt_and_its_decoded_tail(device, case, dtype):
    """420 tokens, the last 40 one by one: every position against the plain implementation; the kept tokens are hundreds of
    positions back, the slow channels still hold what was written there."""
    ids, want = wanted(case, 420, 77)
    runner = make_runner(cases.CASES[case], weights_of(case), dtype, device, num_pages=48)
    got = helpers.replay(runner, helpers.trace_tail_decoded({"far": ids}, tail=40))
    check_rows(got, {"far": want}, dtype, "a long prompt and its tail")


def mid_config():
    first = [cases.latent(8, 48, 24, 40, 96, 120, 70, cases.dense(320)),
             cases.attention(8, 2, 80, 96, (100, 9), cases.moe(192, 16, 2), rot=64, base=1e4, softcap=20.0),
             cases.delta(4, 2, 48, 56, 4, cases.moe(192, 16, 2))]
    return cases.config(first + [cases.again(first, 1), cases.again(first, 0)], width=224, vocab=2000, mult=0.35)


MID = mid_config()


@functools.lru_cache(maxsize=None)
def wider_model():
    weights = cases.make_weights(MID, seed=99, ranks=(40, 24))
    return weights, {name: cases.safe_sequence(MID, weights, n, seed)
                     for name, n, seed in (("far", 300, 5), ("mid", 150, 6), ("short", 70, 7))}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_wider_model_with_pages_of_64(device, dtype):
    """Sizes nearer a real model's over pages of 64: a prompt of 300 with its decoded tail, then three requests in portions beside
    single tokens over four slots and just enough pages."""
    weights, seqs = wider_model()
    runner = make_runner(MID, weights, dtype, device, num_pages=12, page_size=64)
    got = helpers.replay(runner, helpers.trace_tail_decoded({"far": seqs["far"][0]}, tail=40))
    check_rows(got, {"far": seqs["far"][1]}, dtype, "a wider model: prompt and tail")
    got = helpers.replay(runner, helpers.trace_mixed({n: ids for n, (ids, _) in seqs.items()}, seed=3))
    check_rows(got, {n: rows for n, (_, rows) in seqs.items()}, dtype, "a wider model: mixed")
    assert all(g.pool.num_used == 0 for g in runner.cache.groups)


def check_greedy(case, weights, prompts, outs, new, dtype):
    """Every token is the plain implementation's greedy choice for the same prefix (or, in bfloat16, within rounding)."""
    cfg = cases.CASES[case]
    slack = 1e-4 if dtype == "float32" else 0.15
    w64 = {n: t.double() for n, t in weights.items()}
    close = 0
    for prompt, out in zip(prompts, outs):
        ids = out.generated_token_ids()
        assert len(ids) == new
        margins = [math.inf]
        logits = plain.forward(cfg, w64, prompt + ids, margins=margins)[0]
        if margins[0] < (1e-4 if dtype == "float32" else cases.CLOSE_CALL):
            close += 1  # a router's choice that rounding can turn somewhere in this sequence: nothing to compare
            continue
        for i, tok in enumerate(ids):
            row = logits[len(prompt) + i - 1]
            assert row[tok] >= row.max() - slack * float(row.std()), (dtype, len(prompt), i, tok, int(row.argmax()))
    assert close < len(prompts) if dtype == "float32" else True


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(device, tmp_path, dtype):
    """A folder of the design through ``Engine.generate``: scheduler, portions, sampling on the device."""
    from ferrisinfer_b200 import SamplingParams
    from ferrisinfer_b200.engine.engine import Engine
    from ferrisinfer_b200.engine.scheduler import SchedulerConfig

    case = "A"
    weights = weights_of(case)
    engine = Engine(make_folder(tmp_path, cases.CASES[case], weights), dtype=dtype, page_size=16, num_pages=40,
                    scheduler=SchedulerConfig(max_batch_size=4, max_prefill_chunk_tokens=32, max_prefill_batch_tokens=48,
                                              max_sequence_length=256))
    prompts = [cases.random_ids(cases.CASES[case]["vocab"], n, n) for n in (5, 70, 33, 1, 90, 12)]
    outs = engine.generate(prompts, SamplingParams.greedy(max_new_tokens=20))
    check_greedy(case, weights, prompts, outs, 20, dtype)
    assert all(g.pool.num_used == 0 for g in engine.runner.cache.groups)


def test_shared_prompts_where_every_key_stays(device, tmp_path):
    """A model without masks and recurrences: the second request borrows the pages of the first one's prompt."""
    from ferrisinfer_b200 import SamplingParams
    from ferrisinfer_b200.engine.engine import Engine
    from ferrisinfer_b200.engine.scheduler import SchedulerConfig

    case = "E"
    weights = weights_of(case)
    engine = Engine(make_folder(tmp_path, cases.CASES[case], weights), dtype="float32", page_size=8, num_pages=60,
                    scheduler=SchedulerConfig(max_batch_size=4, max_sequence_length=256, min_prefix_share_tokens=8))
    common = cases.random_ids(75, 50, 1)
    prompts = [common + cases.random_ids(75, 9, 2), common + cases.random_ids(75, 17, 3)]
    outs = [engine.generate(p, SamplingParams.greedy(max_new_tokens=12)) for p in prompts]
    assert outs[1].reused_prompt_tokens == 48
    check_greedy(case, weights, prompts, outs, 12, "float32")


def test_a_random_folder_of_the_design_loads_and_generates(device, tmp_path):
    from ferrisinfer_b200 import SamplingParams
    from ferrisinfer_b200.engine.engine import Engine
    from ferrisinfer_b200.weights import write_model_folder

    folder = write_model_folder(cases.CASES["B"], 5, str(tmp_path / "model"))
    a = Engine(folder, dtype="bfloat16", num_pages=64).generate([[1, 2, 3, 4]], SamplingParams.greedy(max_new_tokens=8))
    b = Engine(config=cases.CASES["B"], seed=5, dtype="bfloat16").generate([[1, 2, 3, 4]], SamplingParams.greedy(max_new_tokens=8))
    assert a[0].generated_token_ids() == b[0].generated_token_ids() and len(a[0].generated_tokens) == 8


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_through_the_trace_runner(device, tmp_path, dtype):
    """``bin/trace_run`` as a user runs it (a subprocess fed JSON lines, four state slots, just enough pages): a folder
    of the design is chosen by its config.json, and a mixed schedule over six requests gives the plain logits."""
    from test_trace_run_gpu import run_trace

    case = "B"
    folder = make_folder(tmp_path, cases.CASES[case], weights_of(case))
    lengths = {"a": (70, 31), "b": (33, 32), "c": (101, 33), "d": (48, 34), "e": (64, 35), "f": (90, 36)}
    reqs = requests_of(case, list(lengths), lengths)
    steps = helpers.trace_mixed(reqs, seed=2)
    got = run_trace(folder, dtype, steps, tmp_path / "out", helpers.tokens_held(steps), cases.CASES[case]["vocab"])
    check_rows(got, rows_of(case, list(lengths), lengths), dtype, "the trace runner")


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8, 9, 10])
def test_random_configuration_in_every_way_of_cutting(device, seed):
    """Configurations drawn at random (mixers, sizes, head counts and groupings, masks, feed-forwards, layers that run again, pages of
    4 to 32), replayed whole, with a decoded tail, in portions and in mixed batches, in both precisions against the plain
    implementation."""
    rng = random.Random(seed)
    cfg = cases.random_config(rng)
    weights = cases.make_weights(cfg, seed, (rng.choice([1, 7, 16]), rng.choice([3, 8, 20])))
    page = rng.choice([4, 8, 16, 16, 32])
    lengths = [rng.randint(1, 40), rng.randint(20, 140), rng.randint(2, 70), rng.randint(60, 160), rng.randint(1, 20)]
    safe = {f"r{i}": cases.safe_sequence(cfg, weights, n, seed * 10 + i) for i, n in enumerate(lengths)}
    reqs = {rid: s[0] for rid, s in safe.items()}
    want = {rid: s[1] for rid, s in safe.items()}
    traces = {"whole": helpers.trace_whole(reqs), "tail": helpers.trace_tail_decoded(reqs),
              "portions": helpers.trace_portions(reqs), "mixed": helpers.trace_mixed(reqs, seed)}
    for dtype in ("float32", "bfloat16"):
        for kind, steps in traces.items():
            pages = helpers.tokens_held(steps, round_to=page) // page
            runner = make_runner(cfg, weights, dtype, device, num_pages=pages, max_requests=8, page_size=page)
            got = helpers.replay(runner, steps)
            runner.cache.check_invariants()
            assert all(g.pool.num_used == 0 for g in runner.cache.groups)
            check_rows(got, want, dtype, f"{cfg} page {page} {kind}")
