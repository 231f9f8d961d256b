"""The Retezen decoder on the GPU against the plain implementation (``plain_retezen``, float64): each kernel of its
mechanisms alone, then whole models of several small configurations driven through the step function the ways a
server drives it (whole prompts, token by token, portions down to two tokens, mixed batches over pages and slots that
come back), and greedy generation through the engine."""

import functools
import json
import math
import os
import random

import pytest
import torch

import helpers
import plain_retezen as plain
import retezen_cases as cases
from test_netinex_gpu import fake_ctx, paged, tol_of

pytestmark = pytest.mark.gpu
F32, F64, BF16 = torch.float32, torch.float64, torch.bfloat16
DTYPES = {"float32": F32, "bfloat16": BF16}


def _ops():
    from ferrisinfer_b200.kernels import ops
    return ops


def make_runner(cfg, weights, dtype, device, num_pages=24, max_requests=4, graphs=True, page_size=16):
    from ferrisinfer_b200.config import resolve_config
    from ferrisinfer_b200.engine.runner import ModelRunner
    from ferrisinfer_b200.parts import build_model
    from ferrisinfer_b200.weights.loader import bind_tensors

    arch, c = resolve_config(cfg)
    model = build_model(arch.plan(c))
    bind_tensors(model, weights, DTYPES[dtype], device)
    return ModelRunner(model, DTYPES[dtype], device, page_size=page_size, num_pages=num_pages, max_requests=max_requests,
                       cuda_graphs=graphs)


def make_folder(tmp_path, cfg, weights) -> str:
    from ferrisinfer_b200.weights.safetensors_io import write_safetensors

    folder = str(tmp_path / "model")
    os.makedirs(folder)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), weights)
    return folder


@functools.lru_cache(maxsize=None)
def weights_of(case: str):
    return cases.make_weights(cases.CASES[case], seed=sum(map(ord, case)))


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


def rounded(w: dict) -> dict:
    """Weights as a folder stores them (bfloat16), widened again."""
    return {n: t.to(BF16).float() for n, t in w.items()}


# =========================================================================================== each mechanism alone
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [43, 64, 2048])
def test_embedding_with_learned_positions(device, width, dtype):
    torch.manual_seed(width)
    table, pos = torch.randn(50, width).to(dtype), torch.randn(40, width).to(dtype)
    ids, positions = torch.randint(0, 50, (9,), dtype=torch.int32), torch.randint(0, 40, (9,), dtype=torch.int32)
    positions[0], positions[1] = 0, 39
    out = torch.empty(9, width, device=device)
    rows = torch.empty(9, width, dtype=dtype, device=device)
    _ops().embed_positions(table.to(device), pos.to(device), ids.to(device), positions.to(device), out, rows)
    want = table[ids.long()].float() + pos[positions.long()].float()
    assert torch.equal(out.cpu(), want) and torch.equal(rows.cpu(), want.to(dtype))
    _ops().embed_positions(table.to(device), pos.to(device), ids.to(device), positions.to(device), out)
    assert torch.equal(out.cpu(), want)


@pytest.mark.parametrize("T", [1, 7, 300, 1300])
@pytest.mark.parametrize("width", [43, 64, 600, 1024, 1500, 2048, 4096, 5000])
def test_norm_of_a_result_added_into_the_residual(device, width, T):
    """Aligned and odd widths, few rows and many: the sum and its rounded rows; without a result the rows alone."""
    torch.manual_seed(width + T)
    y, h, w = 3.0 * torch.randn(T, width), torch.randn(T, width), 1.0 + 0.2 * torch.randn(width)
    want = h.double() + plain.rms(y.double(), 1e-3) * w.double()
    got, rows = h.to(device), torch.empty(T, width, dtype=BF16, device=device)
    _ops().rmsnorm_add(y.to(device), w.to(device), 1e-3, got, rows)
    assert torch.allclose(got.cpu().double(), want, atol=2e-6, rtol=2e-6)
    assert torch.equal(rows, got.to(BF16))
    alone = h.to(device)
    _ops().rmsnorm_add(y.to(device), w.to(device), 1e-3, alone)
    assert torch.equal(alone, got)
    _ops().rmsnorm_add(None, None, 0.0, alone, rows.zero_())
    assert torch.equal(rows, alone.to(BF16)) and torch.equal(alone, got)


@pytest.mark.parametrize("width", [43, 64, 2048])
@pytest.mark.parametrize("top,ordered,weighted", [(1, False, True), (3, True, False), (4, True, True), (2, False, False)])
def test_results_of_a_mixture_added_on_the_norms_way(device, width, top, ordered, weighted):
    """The rows to norm are sums of rows that stand apart, in an order of their own or not, weighted or not."""
    ops = _ops()
    torch.manual_seed(width + top)
    T, R = 21, 21 * top + (9 if ordered else 0)
    y, h, w = torch.randn(R, width), torch.randn(T, width), 1.0 + 0.2 * torch.randn(width)
    pos = torch.randperm(R)[:T * top].view(T, top) if ordered else torch.arange(T * top).view(T, top)
    f = torch.rand(T, top) if weighted else torch.ones(T, top)
    want = h.double() + plain.rms((f.double().unsqueeze(-1) * y.double()[pos]).sum(1), 1e-4) * w.double()
    got, rows = h.to(device), torch.empty(T, width, dtype=BF16, device=device)
    parts = ops.PairRows(y.to(device), pos.int().to(device) if ordered else None, f.to(device) if weighted else None, top)
    ops.rmsnorm_add(None, w.to(device), 1e-4, got, rows, parts=parts)
    assert torch.allclose(got.cpu().double(), want, atol=3e-6, rtol=3e-6) and torch.equal(rows, got.to(BF16))


def pooled_setup(device, dtype, T, nkv, d, dv, ps, pool, seed):
    """Random keys and values of ``T`` positions in pages out of order, and empty pages for their blocks' means:
    (keys, values, k cache, v cache, table, PooledKeys with everything zero, slot of every position's block or -1)."""
    ops = _ops()
    g = torch.Generator().manual_seed(seed)
    keys, values = torch.randn(T, nkv, d, generator=g).to(dtype), torch.randn(T, nkv, dv, generator=g).to(dtype)
    blocks = -(-T // ps)
    order = torch.randperm(blocks + 2, generator=g).tolist()
    kc = torch.zeros(blocks + 3, nkv, ps, d, dtype=dtype, device=device)
    vc = torch.zeros(blocks + 3, nkv, ps, dv, dtype=dtype, device=device)
    for j in range(T):
        kc[order[j // ps], :, j % ps] = keys[j].to(device)
        vc[order[j // ps], :, j % ps] = values[j].to(device)
    table = torch.tensor([order[:blocks]], dtype=torch.int32, device=device)
    rows = T // pool
    pblocks = max(1, -(-rows // ps))
    porder = torch.randperm(pblocks + 2, generator=g).tolist()
    ptable = torch.tensor([porder[:pblocks]], dtype=torch.int32, device=device)
    pooled = ops.PooledKeys(torch.zeros(pblocks + 3, nkv, ps, d, dtype=dtype, device=device),
                            torch.zeros(pblocks + 3, nkv, ps, dv, dtype=dtype, device=device), ptable, pool)
    slots = torch.tensor([porder[(j // pool) // ps] * ps + (j // pool) % ps if (j + 1) % pool == 0 else -1 for j in range(T)],
                         dtype=torch.int32, device=device)
    return keys, values, kc, vc, table, pooled, slots


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("nkv,d,dv,ps,pool,T", [(2, 32, 24, 16, 5, 90), (3, 15, 9, 16, 40, 130), (1, 64, 64, 4, 1, 30),
                                                 (4, 128, 128, 16, 16, 100), (2, 8, 200, 8, 3, 33)])
def test_means_of_blocks(device, nkv, d, dv, ps, pool, T, dtype):
    """The launch behind a portion, whole and cut so that blocks span portions: every complete block's row holds the means of
    its keys and values, no other row is touched."""
    ops = _ops()
    keys, values, kc, vc, table, pooled, slots = pooled_setup(device, dtype, T, nkv, d, dv, ps, pool, T)
    flat = lambda t: t.cpu().double().permute(0, 2, 1, 3).reshape(-1, nkv, t.shape[-1])
    for cuts in ([T], [7, 2, 1, T - 10]):
        pooled.k.zero_(), pooled.v.zero_()
        pos = 0
        for n in cuts:
            ctx = fake_ctx(device, [n], [pos], [0])
            ops.pool_blocks(kc, vc, pooled, slots[pos:pos + n].contiguous(), table, ctx)
            pos += n
        k, v = flat(pooled.k), flat(pooled.v)
        used = torch.zeros(k.shape[0], dtype=torch.bool)
        for b in range(T // pool):
            s = int(slots[(b + 1) * pool - 1])
            used[s] = True
            want_k = keys[b * pool:(b + 1) * pool].double().mean(0)
            want_v = values[b * pool:(b + 1) * pool].double().mean(0)
            tol = dict(atol=1e-6, rtol=1e-6) if dtype == F32 else dict(atol=2e-3, rtol=5e-3)
            assert torch.allclose(k[s], want_k, **tol) and torch.allclose(v[s], want_v, **tol), b
        assert not k[~used].any() and not v[~used].any()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("nh,nkv,d,dv", [(4, 2, 32, 24), (3, 3, 15, 9), (4, 1, 64, 64), (2, 2, 20, 12), (16, 8, 128, 64),
                                          (48, 4, 128, 128)])
def test_norm_mixing_cache_write_and_means_of_single_tokens(device, nh, nkv, d, dv, dtype):
    """The kernel between the product and attention: values mixed with (or left for) another layer, and, in steps of single
    tokens, the means of the blocks that the tokens complete, bit for bit those of the launch behind a portion."""
    ops = _ops()
    T, ps, pool, eps = 45, 16, 7, 1e-5
    torch.manual_seed(nh * d)
    rows = torch.randn(T, (nh + nkv) * d + nkv * dv).to(dtype)
    qw, kw, lam = 1.0 + 0.2 * torch.randn(nh * d), 1.0 + 0.2 * torch.randn(nkv * d), torch.tensor([0.35])
    other = torch.randn(T, nkv * dv).to(dtype)
    kc, _, table, slots = paged(device, dtype, T, nkv, d, ps, [2, 0, 1])
    vc = torch.zeros(*kc.shape[:3], dv, dtype=dtype, device=device)
    _, _, _, _, _, pooled, pslots = pooled_setup(device, dtype, T, nkv, d, dv, ps, pool, 1)
    ctx = fake_ctx(device, [T], [0], [0])
    args = (nh, nkv, d, dv, qw.to(device), kw.to(device), eps, None)
    # a portion that mixes
    whole = rows.to(device)
    ops.qk_norm_rotary_cache_write(whole, ctx, slots, kc, vc, *args, mixed_values=other.to(device), mix_lambda=lam.to(device))
    ops.pool_blocks(kc, vc, pooled, pslots, table, ctx)
    x = rows.double()
    q = plain.rms(x[:, :nh * d], eps) * qw.double()
    k = plain.rms(x[:, nh * d:(nh + nkv) * d], eps) * kw.double()
    v = plain.mix_values(x[:, (nh + nkv) * d:], other.double(), lam.double())
    slot = slots.cpu().long()
    flat = lambda t: t.cpu().double().permute(0, 2, 1, 3).reshape(-1, nkv * t.shape[-1])
    assert torch.allclose(whole[:, :nh * d].cpu().double(), q, **tol_of(dtype))
    assert torch.allclose(flat(kc)[slot], k, **tol_of(dtype)) and torch.allclose(flat(vc)[slot], v, **tol_of(dtype))
    # the same token by token, with the means on the way
    kc2, vc2 = torch.zeros_like(kc), torch.zeros_like(vc)
    means = ops.PooledKeys(torch.zeros_like(pooled.k), torch.zeros_like(pooled.v), pooled.block_tables, pool)
    for t in range(T):
        one = fake_ctx(device, [1], [t], [0])
        row = rows[t:t + 1].to(device)
        ops.qk_norm_rotary_cache_write(row, one, slots[t:t + 1].contiguous(), kc2, vc2, *args,
                                       mixed_values=other[t:t + 1].to(device), mix_lambda=lam.to(device), pooled=means,
                                       pool_slots=pslots[t:t + 1].contiguous(), block_tables=table)
        assert torch.equal(row[0, :nh * d], whole[t, :nh * d])
    assert torch.equal(kc2, kc) and torch.equal(vc2, vc)
    assert torch.equal(means.k, pooled.k) and torch.equal(means.v, pooled.v) and pooled.k.any()
    # the layer whose values the others mix with leaves them as projected
    left = torch.zeros(T, nkv * dv, dtype=dtype, device=device)
    ops.qk_norm_rotary_cache_write(rows.to(device), ctx, slots, kc, vc, *args, mixed_values=left)
    assert torch.equal(left.cpu(), rows[:, (nh + nkv) * d:])
    assert torch.equal(flat(vc)[slot], rows[:, (nh + nkv) * d:].double())


def attend(ops, form, q, last, T, k, v, table, pooled, nh, nkv, d, dv, window, scale, device):
    """One row of attention for the query of the last position, through one of the kernel's forms."""
    from ferrisinfer_b200.engine.workspace import Workspace

    tiled = form == "tiled"
    ctx = fake_ctx(device, [T], [0], [0]) if tiled else fake_ctx(device, [1], [last], [0])
    rows = q if tiled else q[last:]
    out = torch.empty(rows.shape[0], nh * dv, device=device, dtype=q.dtype)
    extra = dict(max_kv_len=T, workspace=Workspace(device)) if form == "shares" else {}
    ops.paged_attention_simt(rows.contiguous(), out, k, v, table, ctx.token_seq, ctx.positions, nh, nkv, d, window, scale,
                             v_head_dim=dv, max_q_len=T if tiled else 1, pooled=pooled, **extra)
    return out[-1].float().cpu().double().view(nh, dv)


@pytest.mark.parametrize("form,nh,nkv,d,dv", [("single", 4, 2, 32, 24), ("tiled", 4, 2, 32, 24), ("shares", 4, 2, 32, 48),
                                               ("shares", 8, 1, 64, 32), ("single", 3, 3, 15, 9), ("tiled", 2, 2, 64, 64)])
@pytest.mark.parametrize("window,pool,last", [(24, 5, 27), (24, 5, 28), (24, 5, 200), (5, 16, 19), (5, 16, 20), (5, 16, 21),
                                               (1, 3, 50), (1, 3, 51), (1, 3, 52), (19, 1, 64), (16, 16, 31), (16, 16, 47),
                                               (16, 16, 48), (33, 7, 599), (33, 7, 600), (40, 64, 103), (40, 64, 104)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_one_key_stands_out_at_each_edge(device, window, pool, last, form, nh, nkv, d, dv, dtype):
    """One token's or one block's key is made loud in turn: the first and the last position of the window, the position
    just before it (in the cache, seen by nothing), the last block that lies wholly before the window, the block after
    it (written to its page if the prompt has completed it, and not yet seen), block 0 hundreds of positions back.  What is
    seen takes nearly all the weight; what is not must leave the mean over everything visible."""
    ops = _ops()
    torch.manual_seed(window * 1000 + last)
    ps, T = 16, last + 1
    direction = torch.randn(d)
    direction /= direction.norm()
    seen_tokens, seen_blocks = plain.visible(last, {"size": window, "pool": pool})
    values = torch.randn(T, nkv, dv)
    means = torch.stack([values[b * pool:(b + 1) * pool].mean(0) for b in range(T // pool)]) if T >= pool else torch.zeros(0, nkv, dv)
    q = torch.zeros(T, nh * d)
    q[last] = (3.0 * direction).repeat(nh)
    loud = [("token", j) for j in {last, seen_tokens[0], seen_tokens[0] - 1} if j >= 0]
    n = len(seen_blocks)
    loud += [("block", b) for b in {0, n - 1, n} if 0 <= b < T // pool]
    of = torch.arange(nh) // (nh // nkv)
    for what, at in loud:
        _, _, k, v, table, pooled, slots = pooled_setup(device, dtype, T, nkv, d, dv, ps, pool, 5)
        k.zero_()
        order = table[0].tolist()
        for j in range(T):
            v[order[j // ps], :, j % ps] = values[j].to(device)
        for b in range(T // pool):
            s = int(slots[(b + 1) * pool - 1])
            pooled.v[s // ps, :, s % ps] = means[b].to(device)
        if what == "token":
            k[order[at // ps], :, at % ps] = 10.0 * direction.to(device)
            seen = at in seen_tokens
        else:
            s = int(slots[(at + 1) * pool - 1])
            pooled.k[s // ps, :, s % ps] = 10.0 * direction.to(device)
            seen = at in seen_blocks
        got = attend(ops, form, q.to(device, dtype), last, T, k, v, table, pooled, nh, nkv, d, dv, window, 1.0, device)
        if seen:  # exp(30) against exp(0) of the others
            want = (values[at] if what == "token" else means[at]).double()[of]
        else:
            want = torch.cat([values[seen_tokens], means[:n]]).double().mean(0)[of]
        tol = 1e-4 if dtype == F32 else 1.5e-2
        assert torch.allclose(got, want, atol=tol, rtol=tol), (what, at, seen, got[0, :3], want[0, :3])


@pytest.mark.parametrize("nh,nkv,d,dv", [(4, 2, 32, 24), (8, 1, 64, 40), (2, 2, 128, 128), (40, 2, 24, 8), (6, 3, 200, 136),
                                          (16, 4, 128, 128), (3, 3, 8, 256), (48, 1, 16, 16), (4, 4, 64, 64)])
@pytest.mark.parametrize("window,chunk,pool", [(33, 0, 7), (100, 0, 16), (5, 0, 40), (0, 0, None), (37, 0, None), (0, 48, None)])
def test_attention_on_tensor_cores_keeps_the_weights_whole(device, nh, nkv, d, dv, window, chunk, pool):
    """bf16 rows through the tensor-core forms and through the CUDA-core forms (fp32 throughout): the results differ by the
    last rounding only, in portions of several requests (one behind a cached prefix, one of a single token) and in single
    tokens, whole and in shares, with a sink.  The values of neighbours nearly cancel, so that weights rounded to 16 bits
    would be far off."""
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
    pooled = None
    if pool:
        rows = [-(-(-(-(a + b) // pool)) // ps) for a, b in zip(lengths, starts)]
        ptables = torch.full((len(lengths), max(rows)), -1, dtype=torch.int32)
        at = 0
        for i, n in enumerate(rows):
            ptables[i, :n] = torch.arange(at, at + n, dtype=torch.int32)
            at += n
        pooled = ops.PooledKeys(torch.randn(at + 1, nkv, ps, d).to(BF16).to(device),
                                (sign + torch.randn(at + 1, nkv, ps, dv)).to(BF16).to(device), ptables.to(device), pool)
    sink = torch.randn(nh).to(device)
    for q_lens, first in ((lengths, starts), ([1] * 4, [a + b - 1 for a, b in zip(lengths, starts)])):
        ctx = fake_ctx(device, q_lens, first, [0] * 4)
        T = ctx.num_tokens
        q = torch.randn(T, nh * d + 8).to(BF16).to(device)[:, :nh * d]
        outs = []
        for on, extra in ((True, {}), (True, dict(max_kv_len=450, workspace=Workspace(device))), (False, {})):
            out = torch.full((T, nh * dv), 7.0, dtype=BF16, device=device)
            ops.set_attention_rows(on)
            try:
                ops.paged_attention_simt(q, out, kc, vc, tables.to(device), ctx.token_seq, ctx.positions, nh, nkv, d, window,
                                         1.5 / math.sqrt(d), score_slopes=ops.ScoreTerms(sink=sink), v_head_dim=dv,
                                         max_q_len=max(q_lens), chunk=chunk, pooled=pooled, **extra)
            finally:
                ops.set_attention_rows(True)
            outs.append(out.float())
        for got in outs[:2]:
            err = (got - outs[2]).abs()
            assert bool((err <= 0.008 * outs[2].abs() + 2e-3).all()), (max(q_lens), float(err.max()))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("m", [
    cases.layer(4, 2, 32, 24, (24, 5), None)["mixer"], cases.layer(3, 3, 15, 9, (5, 16), None)["mixer"],
    cases.layer(8, 1, 64, 40, (33, 7), None)["mixer"], cases.layer(2, 2, 128, 128, (16, 16), None)["mixer"],
    cases.layer(6, 3, 40, 16, (7, 1), None)["mixer"], cases.layer(4, 4, 16, 32, (20, None), None)["mixer"],
    cases.layer(4, 2, 24, 24, None, None)["mixer"]])
def test_attention_mixer_against_the_plain_mixer(device, m, dtype):
    """The part itself (product, norms, mixing, cache write, means, attention over window and blocks, output product) whole,
    as a portion behind a cached prefix, and token by token, over pages out of order, against the plain mixer."""
    from ferrisinfer_b200.cache.manager import CacheManager
    from ferrisinfer_b200.parts.attention import GroupedQueryAttention
    from ferrisinfer_b200.parts.base import PagedMeta
    from ferrisinfer_b200.parts.plan import PartSpec

    nh, nkv, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    torch.manual_seed(nh * d)
    W, T, ps = 48, 90, 16
    w = rounded({"m.q": torch.randn(nh * d, W) / math.sqrt(W), "m.k": torch.randn(nkv * d, W) / math.sqrt(W),
                 "m.v": torch.randn(nkv * dv, W) / math.sqrt(W), "m.q.norm": 1.0 + 0.1 * torch.randn(nh * d),
                 "m.k.norm": 1.0 + 0.1 * torch.randn(nkv * d), "m.vmix": torch.tensor(0.4),
                 "m.o": torch.randn(W, nh * dv) / math.sqrt(nh * dv)})
    y, first = torch.randn(T, W).to(dtype), torch.randn(T, nkv * dv).to(dtype)
    want = plain.attention(y.double(), {n: t.double() for n, t in w.items()}, "m", m, 1e-5, first_values=first.double())[0]
    mask = m.get("mask") or {}
    part = GroupedQueryAttention(W, nh, nkv, d, PartSpec("none"), window=mask.get("size"), pool=mask.get("pool"),
                                 scale=m["scale"], v_head_dim=dv, qk_norm={"eps": 1e-5}, fp32_weights=True,
                                 tensor_names={n: n for n in "qkvo"}, value_mix={"lambda": "vmix", "role": "mix"})
    part.bind({n: t.to(device, dtype if t.dim() == 2 else F32) for n, t in w.items()}, "m")
    for cuts in ([T], [40, 17] + [1] * 33, [2] * 30 + [1] * 30, [50] + [1] * 40):
        mgr = CacheManager([part.cache_need()], ps, 12, 2, dtype=dtype, device=device)
        mgr.admit("other"), mgr.extend("other", 20), mgr.commit("other", 20), mgr.admit("a")
        pos = 0
        for n in cuts:
            mgr.extend("a", pos + n)
            ctx = fake_ctx(device, [n], [pos], [0], act_dtype=dtype)
            for g in mgr.groups:
                table = mgr.block_table("a", g.gid)
                stride = g.need.stride
                at = lambda p: -1 if (p + 1) % stride else table[p // stride // ps] * ps + p // stride % ps
                ctx.paged[g.gid] = PagedMeta(torch.tensor([table or [-1]], dtype=torch.int32, device=device), torch.tensor(
                    [at(p) for p in range(pos, pos + n)], dtype=torch.int32, device=device), ps)
            ctx.workspace.get("mixed_values", (n, nkv * dv), dtype).copy_(first[pos:pos + n])
            h = torch.ones(n, W, device=device)
            part.forward(y[pos:pos + n].to(device).contiguous(), h, ctx, mgr.layer_caches[0], True, accumulate=False)
            assert torch.allclose(h.cpu().double(), want[pos:pos + n], **tol_of(dtype, 3.0)), (cuts[:2], pos)
            mgr.commit("a", pos + n)
            pos += n


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,W,E,top", [(1, 40, 5, 1), (9, 44, 12, 3), (70, 64, 3, 3), (400, 72, 9, 2), (33, 256, 64, 8)])
def test_sigmoid_router(device, T, W, E, top, dtype):
    """Also logits far up where sigmoids are equal in 32-bit: the choice goes by the logits."""
    ops = _ops()
    torch.manual_seed(T * E)
    x = torch.randn(T, W).to(dtype)
    wr = (3.0 * torch.randn(E, W) / math.sqrt(W)).to(dtype)
    z = x.double() @ wr.double().T
    ids = torch.empty(T, top, dtype=torch.int32, device=device)
    weights = torch.empty(T, top, device=device)
    ops.moe_router(x.to(device), wr.to(device), None, ids, weights, top, sigmoid=True)
    order = torch.argsort(z, dim=-1, descending=True, stable=True)[:, :top]
    assert torch.equal(ids.cpu().long(), order)
    assert torch.allclose(weights.cpu().double(), torch.sigmoid(torch.gather(z, 1, order)), atol=1e-6, rtol=1e-4)
    b = torch.linspace(40.0, 45.0, E, device=device)
    ops.moe_router(torch.zeros(T, W, device=device, dtype=dtype), wr.to(device), b, ids, weights, top, sigmoid=True)
    assert ids[0].tolist() == list(range(E - 1, E - 1 - top, -1)) and bool((weights == 1.0).all())


@pytest.mark.parametrize("dtype,form", [(F32, "few"), (BF16, "few"), (BF16, "sorted"), (F32, "token"), (BF16, "token")])
@pytest.mark.parametrize("T,W,ff,E,top", [(1, 40, 24, 5, 1), (9, 44, 36, 12, 3), (70, 64, 96, 3, 3), (300, 128, 64, 8, 2),
                                           (17, 43, 33, 6, 4), (700, 256, 384, 16, 1)])
def test_weights_on_the_experts_inputs(device, T, W, ff, E, top, dtype, form):
    """Router and experts together through the part in every form (an expert's weights read once for its tokens, a block per
    token, sorted by expert on tensor cores), replacing the rows and adding into them."""
    ops = _ops()
    from ferrisinfer_b200.parts.feed_forward import MixtureOfExperts

    if form == "sorted" and (W % 8 or ff % 8):
        pytest.skip("rows of no multiple of 8 elements are not sorted")
    torch.manual_seed(T + W)
    w = {"m.router": 1.5 * torch.randn(E, W) / math.sqrt(W)}
    for e in range(E):
        w[f"m.e{e}.gate"], w[f"m.e{e}.up"] = 2.0 * torch.randn(ff, W) / math.sqrt(W), torch.randn(ff, W) / math.sqrt(W)
        w[f"m.e{e}.down"] = torch.randn(W, ff) / math.sqrt(ff)
    w = rounded(w)
    y = torch.randn(T, W).to(dtype)
    margins = [math.inf] * T
    want = plain.mixture(y.double(), {n: t.double() for n, t in w.items()}, "m", {"router": {"experts": E, "top": top}}, margins)
    part = MixtureOfExperts(W, ff, E, top, router_bias_name=None, sigmoid_scores=True, input_weights=True)
    part.bind({n: t.to(device, dtype) for n, t in w.items()}, "m")
    was = ops.MOE_GROUPED_MIN_TOKENS, ops.MOE_FEW_MAX_PAIRS
    ops.MOE_GROUPED_MIN_TOKENS = 1 if form == "sorted" else 1 << 30
    ops.MOE_FEW_MAX_PAIRS = 0 if form == "token" else was[1]
    try:
        h = torch.full((T, W), 7.0, device=device)
        ctx = fake_ctx(device, [T], [0], [0], act_dtype=dtype)
        part.forward(y.to(device), h, ctx, accumulate=False)
        sure = torch.tensor([m > 1e-3 for m in margins])  # a choice that a rounding of the sums could turn is not compared
        assert sure.sum() >= T * 0.8
        assert torch.allclose(h.cpu().double()[sure], want[sure], **tol_of(dtype, 3.0))
        part.forward(y.to(device), h, ctx)
        assert torch.allclose(h.cpu().double()[sure], 2.0 * want[sure], **tol_of(dtype, 6.0))
    finally:
        ops.MOE_GROUPED_MIN_TOKENS, ops.MOE_FEW_MAX_PAIRS = was


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
    """The residual stream after every layer, not only the logits."""
    runner = make_runner(cases.CASES[case], weights_of(case), dtype, device, graphs=False)
    ids = wanted(case, *LENGTHS["edge"])[0]
    want = []
    plain.forward(cases.CASES[case], weights_of(case), ids, after_layer=lambda i, x: want.append(x.clone()))
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
    """A long decode: 150 single tokens through recorded steps, over page borders, windows and blocks."""
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
        assert torch.allclose(together[key], row, atol=3e-5, rtol=3e-5), key


def test_pages_that_the_window_has_passed_come_back_while_a_request_decodes(device):
    """A pool far smaller than the request: the pages behind the window carry it on, the blocks' rows stay."""
    case = "A"  # a window of 24
    ids, want = wanted(case, *LENGTHS["long"])
    runner = make_runner(cases.CASES[case], weights_of(case), "float32", device, num_pages=5, max_requests=1)
    got = helpers.replay(runner, helpers.trace_portions({"a": ids}, sizes=(9, 1, 2, 30, 1, 1, 5)))
    check_rows(got, {"a": want}, "float32", "few pages")
    assert all(g.pool.num_used == 0 for g in runner.cache.groups)


def test_pages_used_again_by_the_next_request(device):
    """One slot and just enough pages: the second request takes what the first one left (keys, means), and computes what it
    computes alone."""
    case = "A"
    runner = make_runner(cases.CASES[case], weights_of(case), "float32", device, num_pages=10, max_requests=1)
    names = ["long", "mid"]
    got = helpers.replay(runner, helpers.trace_portions(requests_of(case, names), sizes=(40, 3, 1)))
    check_rows(got, rows_of(case, names), "float32", "pages used again")


@pytest.mark.parametrize("case,dtype", [("A", "float32"), ("A", "bfloat16"), ("C", "float32")])
def test_a_long_prompt_and_its_decoded_tail(device, case, dtype):
    """520 tokens, the last 40 one by one: every position against the plain implementation, blocks hundreds of positions
    back in every logit that is compared."""
    ids, want = wanted(case, 520, 77)
    runner = make_runner(cases.CASES[case], weights_of(case), dtype, device, num_pages=48)
    got = helpers.replay(runner, helpers.trace_tail_decoded({"far": ids}, tail=40))
    check_rows(got, {"far": want}, dtype, "a long prompt and its tail")


MID = cases.config([cases.layer(8, 2, 80, 96, (100, 9), cases.dense(384, 1.5), v_mix=False),
                    cases.layer(8, 2, 80, 96, (100, 9), cases.moe(192, 16, 4)), cases.layer(8, 2, 80, 96, (100, 9), None),
                    cases.layer(8, 2, 80, 96, (100, 9), cases.moe(192, 16, 4))], width=256, vocab=2000, logit_scale=0.4)


@functools.lru_cache(maxsize=None)
def wider_model():
    weights = cases.make_weights(MID, seed=99)
    return weights, {name: cases.safe_sequence(MID, weights, n, seed)
                     for name, n, seed in (("far", 400, 5), ("mid", 150, 6), ("short", 70, 7))}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_wider_model_with_pages_of_64(device, dtype):
    """Sizes nearer a real model's (a width of 256, heads of 80 with values of 96, four of sixteen experts, a vocabulary of
    2,000) over pages of 64: a prompt of 400 with its decoded tail, then three requests in portions beside single tokens
    over four slots and just enough pages."""
    weights, seqs = wider_model()
    runner = make_runner(MID, weights, dtype, device, num_pages=13, page_size=64)
    got = helpers.replay(runner, helpers.trace_tail_decoded({"far": seqs["far"][0]}, tail=40))
    check_rows(got, {"far": seqs["far"][1]}, dtype, "a wider model: prompt and tail")
    got = helpers.replay(runner, helpers.trace_mixed({n: ids for n, (ids, _) in seqs.items()}, seed=3))
    check_rows(got, {n: rows for n, (_, rows) in seqs.items()}, dtype, "a wider model: mixed")
    assert all(g.pool.num_used == 0 for g in runner.cache.groups)


def check_greedy(case, weights, prompts, outs, new, dtype):
    """Every token is the plain implementation's greedy choice for the same prefix (or, in bfloat16, within rounding)."""
    cfg = cases.CASES[case]
    slack = 1e-4 if dtype == "float32" else 0.15
    close = 0
    for prompt, out in zip(prompts, outs):
        ids = out.generated_token_ids()
        assert len(ids) == new
        margins = [math.inf] * (len(prompt) + new)
        logits = plain.forward(cfg, weights, prompt + ids, margins=margins)[0]
        if min(margins) < (1e-4 if dtype == "float32" else cases.CLOSE_CALL):
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
    """A model without masks: the second request borrows the pages of the first one's prompt (mixed values included)."""
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


def test_no_request_grows_beyond_the_position_table(device, tmp_path):
    from ferrisinfer_b200 import SamplingParams
    from ferrisinfer_b200.engine.engine import Engine
    from ferrisinfer_b200.engine.runner import StepEntry
    from ferrisinfer_b200.engine.scheduler import FinishReason
    from ferrisinfer_b200.errors import FerrisError

    cfg = dict(cases.CASE_A, max_positions=40)
    weights = cases.make_weights(cfg, 3)
    engine = Engine(make_folder(tmp_path, cfg, weights), dtype="float32", num_pages=20)
    out = engine.generate(cases.random_ids(97, 30, 1), SamplingParams.greedy(max_new_tokens=64))
    assert out.finish_reason is FinishReason.SEQUENCE_LENGTH and len(out.generated_tokens) == 10
    with pytest.raises(FerrisError):
        engine.runner.step([StepEntry("a", cases.random_ids(97, 41, 1), [])])


def test_a_random_folder_of_the_design_loads_and_generates(device, tmp_path):
    from ferrisinfer_b200 import SamplingParams
    from ferrisinfer_b200.engine.engine import Engine
    from ferrisinfer_b200.weights import write_model_folder

    folder = write_model_folder(cases.CASE_B, 5, str(tmp_path / "model"))
    a = Engine(folder, dtype="bfloat16", num_pages=64).generate([[1, 2, 3, 4]], SamplingParams.greedy(max_new_tokens=8))
    b = Engine(config=cases.CASE_B, seed=5, dtype="bfloat16").generate([[1, 2, 3, 4]], SamplingParams.greedy(max_new_tokens=8))
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


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_random_configuration_in_every_way_of_cutting(device, seed):
    """Configurations drawn at random (sizes, head counts and groupings, masks, mixing, feed-forwards, the number of the
    layers, pages of 4 to 32), replayed whole, with a decoded tail, in portions and in mixed batches, in both precisions
    against the plain implementation."""
    rng = random.Random(seed)
    cfg = cases.random_config(rng)
    weights = cases.make_weights(cfg, seed)
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
