"""Designs side by side at equal layer sizes: the Kugilix decoder beside the Qwen2 dense decoder, or (``design`` =
"nusudra" / "netinex") the Nusudra or the Netinex decoder beside both, or (``design`` = "sumevik") the Sumevik decoder
beside the Netinex decoder (the closest existing design: attention within chunks, a linear recurrence, experts) and
Qwen2, or (``design`` = "retezen") the Retezen decoder beside the same two, or (``design`` = "lukelorn") the Lukelorn decoder
beside the Nusudra decoder (the closest existing design: a delta rule, attention over a latent), Retezen (attention on tensor
cores, experts with weights on their inputs) and Qwen2, random weights.

Called by ``bench.py --designs [--design nusudra|netinex|sumevik|retezen|lukelorn]``.  For each of a few sizes that resemble a real model's layers it measures, through
the step function, the prefill of one prompt and decode steps at two batch sizes for both designs, and times the
kernels that only the Kugilix design has (decayed linear attention, the windowed attention with slopes, the short
convolution, the norms in groups, the gated norm, the activation) alone, with what they reach of the measured copy
bandwidth or, where they are bound by fp32 arithmetic, of the nominal fp32 rate.
"""

from __future__ import annotations

import math
import statistics

FP32_NOMINAL_TFLOPS = 80.0  # B200, fp32 FMAs outside the tensor cores (nominal; there is no measured figure)

SIZES = {
    # name: width, heads, kv heads, head size, feed-forward, layers of the Kugilix model (a span of four runs twice)
    "1B-like": dict(width=2048, heads=16, kv_heads=4, dim=128, ff=8192, layers=8),
    "3B-like": dict(width=3072, heads=24, kv_heads=8, dim=128, ff=12288, layers=8),
    "small": dict(width=1024, heads=16, kv_heads=8, dim=64, ff=4096, layers=8),
}
WINDOW = 1024
VOCAB = 32000


def kugilix_config(s: dict) -> dict:
    att = {"type": "attention",
           "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"],
                     "scale": 1.0 / math.sqrt(s["dim"]), "mask": {"size": WINDOW}, "q_temp": {"coef": 0.3, "every": 128}},
           "mlp": {"kind": "dense", "ff": s["ff"]}}
    lin = {"type": "lightning",
           "mixer": {"heads": s["heads"], "dim": s["dim"], "vdim": s["dim"],
                     "decay": [round(1.0 - 2.0 ** (-2 - 6 * h / s["heads"]), 6) for h in range(s["heads"])]},
           "mlp": {"kind": "dense", "ff": s["ff"]}}
    order = [att, lin, lin, att, lin, lin, att, lin]
    layers = [order[i % len(order)] for i in range(s["layers"])]
    return {"architecture": "Kugilix", "vocab": VOCAB, "width": s["width"], "embedding": {"scale": math.sqrt(s["width"])},
            "norm": {"eps": 1e-6, "groups": 4}, "canon": {"taps": 4}, "layers": layers,
            "loop": {"start": 2, "stop": 6, "times": 2}}


def kugilix_runs(s: dict) -> int:
    return s["layers"] + 4


def qwen2_config(s: dict) -> dict:
    """The closest existing design with as many layer runs, the same width and heads, and a gated feed-forward of as
    many weights as the plain one (three matrices of 2/3 the width), every layer over the same window."""
    inter = (2 * s["ff"] // 3 + 127) // 128 * 128
    n = kugilix_runs(s)
    return {"architectures": ["Qwen2ForCausalLM"], "model_type": "qwen2", "vocab_size": VOCAB, "hidden_size": s["width"],
            "intermediate_size": inter, "num_hidden_layers": n, "num_attention_heads": s["heads"],
            "num_key_value_heads": s["kv_heads"], "head_dim": s["dim"], "max_position_embeddings": 8192,
            "rms_norm_eps": 1e-6, "rope_theta": 1e6, "hidden_act": "silu", "tie_word_embeddings": False,
            "use_sliding_window": True, "sliding_window": WINDOW, "max_window_layers": 0}


NUSUDRA_ORDER = ("delta", "latent_attention", "parallel")


def nusudra_config(s: dict) -> dict:
    """As many layers as the Kugilix model has layer runs, its three mixers in turn; the same width, heads, head
    size and feed-forward; four residual streams.  The latent row (192 + 64) is the widest the general attention
    kernel takes; the state-space layer has as many heads of the same size, a state of 128 and one group."""
    H, G, d = s["heads"], s["kv_heads"], s["dim"]
    mixers = {
        "delta": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "conv": 4},
        "latent_attention": {"heads": H, "dim": d, "rot_dim": 64, "vdim": d, "kv_rank": 192,
                             "scale": 1.0 / math.sqrt(d + 64), "rot": {"base": 10000.0, "dims": 64}},
        "parallel": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": 1.0 / math.sqrt(d)},
                     "right": {"heads": H, "vdim": d, "state": 128, "groups": 1, "norm_groups": 1, "conv": 4}},
    }
    layers = [{"type": NUSUDRA_ORDER[i % 3], "mixer": mixers[NUSUDRA_ORDER[i % 3]], "mlp": {"kind": "dense", "ff": s["ff"]}}
              for i in range(kugilix_runs(s))]
    return {"architecture": "Nusudra", "vocab": VOCAB, "width": s["width"], "embedding": {"scale": math.sqrt(s["width"])},
            "norm": {"eps": 1e-6}, "streams": 4, "layers": layers}


EXPERTS, TOP = 8, 2


def netinex_expert_ff(s: dict) -> int:
    """An expert's inner size such that the ``TOP`` experts a token uses hold as many weights as the Kugilix model's
    plain feed-forward (two matrices of ff against TOP x three), in multiples of 64."""
    return max(64, (2 * s["ff"]) // (3 * TOP) // 64 * 64)


def netinex_config(s: dict) -> dict:
    """As many layers as the Kugilix model has layer runs, in its order (an attention, two retentions, ...); the same
    width, heads, head size; chunks as long as the other designs' window; ``TOP`` of ``EXPERTS`` gated experts that
    together hold the weights of the plain feed-forward."""
    H, G, d = s["heads"], s["kv_heads"], s["dim"]
    mlp = {"kind": "moe", "expert": {"ff": netinex_expert_ff(s)}, "router": {"experts": EXPERTS, "top": TOP}}
    att = {"type": "attention",
           "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": 1.0 / math.sqrt(d), "mask": {"size": WINDOW},
                     "rot": {"base": 10000.0, "dims": d,
                             "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}},
           "mlp": mlp}
    ret = {"type": "retention",
           "mixer": {"heads": H, "dim": d, "vdim": d, "rot": {"base": 1000000.0, "dims": d},
                     "decay": [round(1.0 - 2.0 ** (-2 - 6 * h / H), 6) for h in range(H)]},
           "mlp": mlp}
    order = [att, ret, ret]
    return {"architecture": "Netinex", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
            "layers": [order[i % 3] for i in range(kugilix_runs(s))]}


SUMEVIK_IDENTITY = 2  # router outputs beside the EXPERTS experts that stand for "the token's own row"


def sumevik_dense_ff(s: dict) -> int:
    """The inner size of a gated feed-forward of as many weights as the plain one of ``ff`` (three matrices for two)."""
    return (2 * s["ff"] // 3 + 127) // 128 * 128


def sumevik_config(s: dict) -> dict:
    """As many layers as the Kugilix model has layer runs: two recurrent layers, then an attention beside a gated linear
    attention, and so on; the recurrence as wide as the model with as many gate blocks as heads; the same heads and head
    size, chunks as long as the other designs' window, half of every head rotating; the linear attention with as many
    heads, keys of half and values of the full head size; a gated feed-forward in every second layer, ``TOP`` of
    ``EXPERTS`` experts (+ ``SUMEVIK_IDENTITY`` identity experts, two groups of which one stays) in the others."""
    H, G, d, W = s["heads"], s["kv_heads"], s["dim"], s["width"]
    outputs = EXPERTS + SUMEVIK_IDENTITY
    moe = {"kind": "moe", "expert": {"ff": netinex_expert_ff(s), "limit": 7.0},
           "router": {"experts": EXPERTS, "identity": SUMEVIK_IDENTITY, "top": TOP, "groups": {"count": 2, "keep": 1}}}
    assert outputs % 2 == 0
    dense = {"kind": "dense", "ff": sumevik_dense_ff(s)}
    rec = {"type": "rglru", "mixer": {"width": W, "blocks": H, "conv": 4}}
    par = {"type": "parallel",
           "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": 1.0 / math.sqrt(d),
                              "mask": {"size": WINDOW}, "rot": {"base": 500000.0, "dims": d // 2}},
                     "right": {"heads": H, "dim": d // 2, "vdim": d, "tau": 8.0}, "left_scale": 0.9, "right_scale": 1.2}}
    order = [rec, rec, par]
    layers = [dict(order[i % 3], mlp=moe if i % 2 else dense) for i in range(kugilix_runs(s))]
    return {"architecture": "Sumevik", "vocab": VOCAB, "width": W, "norm": {"eps": 1e-6}, "logit_scale": 0.7, "layers": layers}


RETEZEN_POOL = 16  # positions to a pooled block


def retezen_config(s: dict) -> dict:
    """As many layers as the Kugilix model has layer runs, all of them attention; the same width, heads, head size; a window
    as long as the other designs' with blocks of ``RETEZEN_POOL`` before it; values mixed from the second layer on; a gated
    feed-forward of as many weights as the plain one in the first layer, ``TOP`` of ``EXPERTS`` experts in the others."""
    H, G, d = s["heads"], s["kv_heads"], s["dim"]
    mixer = {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": 1.0 / math.sqrt(d), "v_mix": True,
             "mask": {"size": WINDOW, "pool": RETEZEN_POOL}}
    moe = {"kind": "moe", "expert": {"ff": netinex_expert_ff(s)}, "router": {"experts": EXPERTS, "top": TOP}}
    dense = {"kind": "dense", "ff": sumevik_dense_ff(s), "limit": 7.0}
    return {"architecture": "Retezen", "vocab": VOCAB, "width": s["width"], "max_positions": 8192, "norm": {"eps": 1e-6},
            "logit_scale": 0.7, "layers": [{"type": "attention", "mixer": mixer, "mlp": moe if i else dense}
                                           for i in range(kugilix_runs(s))]}


LUKELORN_KEEP = 64  # first tokens that stay visible beside the window
LUKELORN_ORDER = ("latent_attention", "attention", "channel_delta")


def lukelorn_expert_ff(s: dict) -> int:
    """An expert's inner size such that the ``TOP`` experts a token uses hold as many weights as the plain feed-forward."""
    return s["ff"] // TOP


def lukelorn_q_rank(s: dict) -> int:
    return 3 * s["width"] // 8


def lukelorn_config(s: dict) -> dict:
    """As many layers as the Kugilix model has layer runs, its three mixers in turn; the same width, heads, head size; windows
    as long as the other designs'; the latent row of the Nusudra model (192 + 64), queries through a latent of three eighths of
    the width; a gated feed-forward of as many weights as the plain one in the first layer, ``TOP`` of ``EXPERTS`` experts in
    the others; no layer's tensors run twice."""
    H, G, d = s["heads"], s["kv_heads"], s["dim"]
    mixers = {
        "latent_attention": {"heads": H, "dim": d, "rot_dim": 64, "vdim": d, "q_rank": lukelorn_q_rank(s), "kv_rank": 192,
                             "scale": 1.0 / math.sqrt(d + 64), "rot": {"base": 1e6, "dims": 64}, "mask": {"size": WINDOW}},
        "attention": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": 1.0 / math.sqrt(d), "softcap": 50.0,
                      "rot": {"base": 5e5, "dims": d, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 2048}},
                      "mask": {"size": WINDOW, "keep_first": LUKELORN_KEEP}},
        "channel_delta": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "conv": 4},
    }
    moe = {"kind": "moe", "expert": {"ff": lukelorn_expert_ff(s)}, "router": {"experts": EXPERTS, "top": TOP}}
    dense = {"kind": "dense", "ff": sumevik_dense_ff(s)}
    layers = [{"type": LUKELORN_ORDER[i % 3], "mixer": mixers[LUKELORN_ORDER[i % 3]], "mlp": moe if i else dense}
              for i in range(kugilix_runs(s))]
    return {"architecture": "Lukelorn", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-6}, "residual_mult": 0.5,
            "layers": layers}


def _timed(fn, flush, warmup=3, iters=5, reps=1):
    """Seconds per launch: the median of ``iters`` regions of ``reps`` launches back to back, a buffer larger than L2
    written before each region.  ``reps`` > 1 for kernels of a few microseconds, whose single launch would be timed
    together with the host's way to it; their operands are small and lie in L2 inside a step as well."""
    import torch

    for _ in range(warmup):
        fn()
    times = []
    for _ in range(iters):
        flush.add_(1.0)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(reps):
            fn()
        e1.record()
        torch.cuda.synchronize()
        times.append(e0.elapsed_time(e1) / reps)
    return statistics.median(times) * 1e-3


def kernel_numbers(s: dict, peaks: dict) -> dict:
    """The Kugilix design's own kernels alone at the layer sizes ``s``: seconds, and the fraction of the roofline each
    is measured against (``hbm``: bytes that must move over the measured copy bandwidth; ``fp32``: FMAs over the
    nominal fp32 rate)."""
    import torch
    from types import SimpleNamespace

    from ferrisinfer_b200.kernels import ops
    from ferrisinfer_b200.parts.position import DistanceSlopes

    dev = torch.device("cuda")
    bf = torch.bfloat16
    flush = torch.zeros(96 << 20, dtype=torch.float32, device=dev)  # 384 MB
    W, H, G, d, ff = s["width"], s["heads"], s["kv_heads"], s["dim"], s["ff"]
    hbm = peaks["hbm_gbs"] * 1e9
    out = {}

    def ctx_of(q_lens, start):
        S = len(q_lens)
        q_start = [0]
        for n in q_lens:
            q_start.append(q_start[-1] + n)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        return SimpleNamespace(num_tokens=q_start[-1], num_seqs=S, max_q_len=max(q_lens), workspace=None,
                               token_seq=i32([i for i in range(S) for _ in range(q_lens[i])]),
                               positions=i32([start + j for i in range(S) for j in range(q_lens[i])]),
                               seq_q_start=i32(q_start), seq_start_pos=i32([start] * S), seq_state_slot=i32(list(range(S))))

    def record(name, seconds, bytes_=None, flops=None):
        e = {"us": round(seconds * 1e6, 1)}
        if bytes_ is not None:
            e["GBps"] = round(bytes_ / seconds / 1e9, 1)
            e["frac_hbm"] = round(bytes_ / seconds / hbm, 3)
        if flops is not None:
            e["TFLOPs_fp32"] = round(flops / seconds / 1e12, 2)
            e["frac_fp32_nominal"] = round(flops / seconds / (FP32_NOMINAL_TFLOPS * 1e12), 3)
        out[name] = e

    # ---- decayed linear attention
    for name, q_lens in (("linear_attention_decode_b64", [1] * 64), ("linear_attention_prefill_2048", [2048])):
        T, S = sum(q_lens), len(q_lens)
        proj = torch.randn(T, 4 * H * d, device=dev).to(bf)
        state = torch.zeros(S + 1, H, d, d, device=dev)
        o = torch.empty(T, H * d, device=dev)
        decay = torch.full((H,), 0.97, device=dev)
        ctx = ctx_of(q_lens, 0)
        t = _timed(lambda: ops.linear_attention(proj, (0, H * d, 2 * H * d), o, state, decay, ctx, H, d, d, silu=True), flush)
        moved = 2 * S * H * d * d * 4 + T * 3 * H * d * 2 + T * H * d * 4
        record(name, t, bytes_=moved, flops=4.0 * T * H * d * d)
    # ---- windowed attention with unit-norm keys and slopes
    slopes = DistanceSlopes(8.0).score_slopes(H, dev)
    for name, batch, q_len, ctx_len in (("window_attention_decode_b64", 64, 1, 2048), ("window_attention_prefill_2048", 1, 2048, 0)):
        T = batch * q_len
        pages_each = (ctx_len + q_len + 15) // 16
        k = torch.randn(batch * pages_each + 1, G, 16, d, device=dev).to(bf)
        v = torch.randn_like(k)
        tables = torch.arange(batch * pages_each, dtype=torch.int32, device=dev).view(batch, pages_each)
        qkv = torch.randn(T, (H + 2 * G) * d, device=dev).to(bf)
        o = torch.empty(T, H * d, dtype=bf, device=dev)
        ctx = ctx_of([q_len] * batch, ctx_len)
        t = _timed(lambda: ops.paged_attention_simt(qkv, o, k, v, tables, ctx.token_seq, ctx.positions, H, G, d, WINDOW,
                                                    1.0 / math.sqrt(d), score_slopes=slopes, v_head_dim=d,
                                                    max_q_len=q_len), flush)
        keys = sum(min(WINDOW, ctx_len + j + 1) for j in range(q_len)) * batch
        if q_len == 1:
            record(name, t, bytes_=batch * G * min(WINDOW, ctx_len + 1) * 2 * d * 2 + T * H * d * 4, flops=4.0 * keys * H * d)
        else:
            record(name, t, flops=4.0 * keys * H * d)
        slots = (tables[ctx.token_seq.long(), (ctx.positions // 16).long()] * 16 + ctx.positions % 16).int()
        t = _timed(lambda: ops.qk_prepare_cache_write(qkv, ctx.positions, slots, k, v, H, G, d, d, 1e-6, (0.3, 128)), flush,
                   reps=10)
        record(name.replace("window_attention", "qk_prepare"), t, bytes_=T * (2 * H * d + 4 * G * d) * 2)
    # ---- row-wise kernels of a long step and of a decode step
    for tag, T in (("2048", 2048), ("b64", 64)):
        h = torch.randn(T, W, device=dev)
        w1, w2 = torch.ones(W, device=dev), torch.ones(W, device=dev)
        a, b = torch.empty(T, W, dtype=bf, device=dev), torch.empty(T, W, dtype=bf, device=dev)
        t = _timed(lambda: ops.grouped_rmsnorm_pair(h, w1, w2, 1e-6, 4, a, b), flush, reps=10 if T <= 64 else 1)
        record(f"norm_pair_{tag}", t, bytes_=T * W * (4 + 2 + 2))
        cw = torch.randn(W, 4, device=dev) * 0.1
        cs = torch.zeros(T + 1, 3, W, device=dev)
        ctx = ctx_of([T], 0) if T > 64 else ctx_of([1] * T, 5)
        t = _timed(lambda: ops.short_conv(a, b, cw, cs, ctx), flush, reps=10 if T <= 64 else 1)
        record(f"short_conv_{tag}", t, bytes_=T * W * 4 + (ctx.num_seqs * 3 * W * 8 if T <= 64 else 0))
        z = torch.randn(T, ff, device=dev).to(bf)
        pq = torch.tensor([0.3, -0.2], device=dev)
        t = _timed(lambda: ops.activation(z, z, "xielu", pq), flush, reps=10 if T <= 64 else 1)
        record(f"xielu_{tag}", t, bytes_=T * ff * 4)
        o = torch.randn(T, H * d, device=dev)
        g = torch.randn(T, H * d, device=dev).to(bf)
        y = torch.empty(T, H * d, dtype=bf, device=dev)
        nw = torch.ones(H * d, device=dev)
        t = _timed(lambda: ops.gated_rmsnorm(o, g, nw, 1e-6, y), flush, reps=10 if T <= 64 else 1)
        record(f"gated_norm_{tag}", t, bytes_=T * H * d * (4 + 2 + 2))
    return out


def nusudra_kernel_numbers(s: dict, peaks: dict) -> dict:
    """The Nusudra design's own kernels alone at the layer sizes ``s``, measured as ``kernel_numbers`` measures."""
    import torch
    from types import SimpleNamespace

    from ferrisinfer_b200.engine.workspace import Workspace
    from ferrisinfer_b200.kernels import ops

    dev = torch.device("cuda")
    bf = torch.bfloat16
    flush = torch.zeros(96 << 20, dtype=torch.float32, device=dev)  # 384 MB
    W, H, G, d = s["width"], s["heads"], s["kv_heads"], s["dim"]
    hbm = peaks["hbm_gbs"] * 1e9
    ws = Workspace(dev)
    out = {}

    def ctx_of(q_lens, start):
        S = len(q_lens)
        q_start = [0]
        for n in q_lens:
            q_start.append(q_start[-1] + n)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        return SimpleNamespace(num_tokens=q_start[-1], num_seqs=S, max_q_len=max(q_lens), workspace=ws,
                               max_kv_len=start + max(q_lens),
                               token_seq=i32([i for i in range(S) for _ in range(q_lens[i])]),
                               positions=i32([start + j for i in range(S) for j in range(q_lens[i])]),
                               seq_q_start=i32(q_start), seq_start_pos=i32([start] * S), seq_state_slot=i32(list(range(S))))

    def record(name, seconds, bytes_=None, flops=None):
        e = {"us": round(seconds * 1e6, 1)}
        if bytes_ is not None:
            e["GBps"] = round(bytes_ / seconds / 1e9, 1)
            e["frac_hbm"] = round(bytes_ / seconds / hbm, 3)
        if flops is not None:
            e["TFLOPs_fp32"] = round(flops / seconds / 1e12, 2)
            e["frac_fp32_nominal"] = round(flops / seconds / (FP32_NOMINAL_TFLOPS * 1e12), 3)
        out[name] = e

    # ---- the recurrences: delta rule (q/k heads shared by heads / G value heads) and the state-space form (state 128)
    for form, qk_heads, n, delta in (("delta_rule", G, d, True), ("state_space", 1, 128, False)):
        for tag, q_lens in (("decode_b64", [1] * 64), ("prefill_2048", [2048])):
            T, S = sum(q_lens), len(q_lens)
            q = (torch.randn(T, qk_heads * n, device=dev) / math.sqrt(n)).to(bf)
            k = (torch.randn(T, qk_heads * n, device=dev) / math.sqrt(n)).to(bf)
            v = torch.randn(T, H * d, device=dev).to(bf)
            decay, beta = torch.full((T, H), 0.97, device=dev), torch.full((T, H), 0.5, device=dev)
            state = torch.zeros(S + 1, H, d, n, device=dev)
            o = torch.empty(T, H * d, device=dev)
            ctx = ctx_of(q_lens, 0)
            t = _timed(lambda: ops.gated_recurrence(q, k, v, decay, beta, o, state, ctx, H, qk_heads, n, d, delta_rule=delta), flush)
            moved = 2 * S * H * n * d * 4 + T * (2 * qk_heads * n + H * d) * 2 + T * H * d * 4
            record(f"{form}_{tag}", t, bytes_=moved, flops=(6.0 if delta else 4.0) * T * H * n * d)
    # ---- attention with a sink and a logarithmic distance penalty (every key is seen), and over the shared latent
    terms = ops.ScoreTerms(log_r1=torch.full((H,), 0.5, device=dev), log_r2=torch.full((H,), 0.3, device=dev),
                           sink=torch.zeros(H, device=dev))
    rank, rot = 192, 64
    for name, batch, q_len, ctx_len in (("decode_b64", 64, 1, 2048), ("prefill_2048", 1, 2048, 0)):
        T = batch * q_len
        pages_each = (ctx_len + q_len + 15) // 16
        tables = torch.arange(batch * pages_each, dtype=torch.int32, device=dev).view(batch, pages_each)
        ctx = ctx_of([q_len] * batch, ctx_len)
        keys = sum(ctx_len + j + 1 for j in range(q_len)) * batch
        k = torch.randn(batch * pages_each + 1, G, 16, d, device=dev).to(bf)
        v = torch.randn_like(k)
        qkv = torch.randn(T, (H + 2 * G) * d, device=dev).to(bf)
        o = torch.empty(T, H * d, dtype=bf, device=dev)
        t = _timed(lambda: ops.paged_attention_simt(qkv, o, k, v, tables, ctx.token_seq, ctx.positions, H, G, d, 0,
                                                    1.0 / math.sqrt(d), score_slopes=terms, v_head_dim=d, max_q_len=q_len,
                                                    max_kv_len=ctx_len + q_len, workspace=ws), flush)
        record(f"sink_attention_{name}", t, flops=4.0 * keys * H * d,
               bytes_=batch * G * (ctx_len + 1) * 2 * d * 2 + T * H * d * 4 if q_len == 1 else None)
        kl = torch.randn(batch * pages_each + 1, 1, 16, rank + rot, device=dev).to(bf)
        ql = torch.randn(T, H * (rank + rot), device=dev).to(bf)
        ol = torch.empty(T, H * rank, dtype=bf, device=dev)
        t = _timed(lambda: ops.paged_attention_simt(ql, ol, kl, None, tables, ctx.token_seq, ctx.positions, H, 1, rank + rot, 0,
                                                    0.07, v_head_dim=rank, max_q_len=q_len, max_kv_len=ctx_len + q_len,
                                                    workspace=ws, values_in_keys=True), flush)
        record(f"latent_attention_{name}", t, flops=2.0 * keys * H * (2 * rank + rot),
               bytes_=batch * (ctx_len + 1) * (rank + rot) * 2 + T * H * (2 * rank + rot) * 2 if q_len == 1 else None)
        # the per-head products around it: plain queries through the key up-projection, latents through the value one
        x = torch.randn(T, H * (d + rot), device=dev).to(bf)
        uk = (torch.randn(H, d, rank, device=dev) / math.sqrt(d)).to(bf)
        t = _timed(lambda: ops.head_gemm(x, d + rot, uk, ql, rank + rot), flush, reps=10 if T <= 64 else 1)
        record(f"head_product_{name}", t, flops=2.0 * T * H * d * rank, bytes_=H * d * rank * 2 + T * H * (d + rank) * 2)
        proj = torch.randn(T, H * (d + rot) + rank + rot, device=dev).to(bf)
        slots = (tables[ctx.token_seq.long(), (ctx.positions // 16).long()] * 16 + ctx.positions % 16).int()
        freq = torch.full((rot // 2,), 0.01, device=dev)
        nw = torch.ones(rank, device=dev)
        qw, table = H * (d + rot), ops.RotaryTable(freq, rot)
        t = _timed(lambda: ops.latent_prepare(ctx.positions, table, 1e-6, H, d, rot, rank, queries=(proj[:, :qw], ql),
                                              keys=(proj[:, qw:], nw, slots, kl)), flush, reps=10 if T <= 64 else 1)
        record(f"latent_prepare_{name}", t, bytes_=T * (2 * H * rot + 2 * (rank + rot)) * 2)
    # ---- row-wise kernels of a long step and of a decode step
    S4 = 4
    for tag, T in (("2048", 2048), ("b64", 64)):
        xs = torch.randn(T, S4 * W, device=dev)
        y = torch.randn(T, W, device=dev)
        mix, ow, iw, nw = torch.eye(S4, device=dev), torch.ones(S4, device=dev), torch.full((S4,), 0.25, device=dev), torch.ones(W, device=dev)
        a, b = torch.empty(T, W, dtype=bf, device=dev), torch.empty(T, W, dtype=bf, device=dev)
        reps = 10 if T <= 64 else 1
        t = _timed(lambda: ops.streams_step(xs, S4, write=(y, mix, ow), read=(iw, nw, 1e-6, a)), flush, reps=reps)
        record(f"streams_write_read_{tag}", t, bytes_=T * W * (2 * S4 * 4 + 4 + 2))
        ctx = ctx_of([T], 0) if T > 64 else ctx_of([1] * T, 5)
        st = torch.zeros(T + 1, W, device=dev)
        sh = torch.full((W,), 0.3, device=dev)
        t = _timed(lambda: ops.token_shift(a, b, sh, st, ctx), flush, reps=reps)
        record(f"token_shift_{tag}", t, bytes_=T * W * 4 + (T * W * 8 if T <= 64 else 0))
        C = (2 * G + H) * d
        wide = torch.randn(T, C + 64, device=dev).to(bf)
        conv = torch.empty(T, C, dtype=bf, device=dev)
        cw = torch.randn(C, 4, device=dev) * 0.1
        cs = torch.zeros(T + 1, 3, C, device=dev)
        t = _timed(lambda: ops.short_conv(wide[:, :C], conv, cw, cs, ctx, residual=False, silu=True), flush, reps=reps)
        record(f"conv_silu_{tag}", t, bytes_=T * C * 4 + (ctx.num_seqs * 3 * C * 8 if T <= 64 else 0))
        o = torch.randn(T, H * d, device=dev)
        g = torch.randn(T, H * d, device=dev).to(bf)
        yy = torch.empty(T, H * d, dtype=bf, device=dev)
        t = _timed(lambda: ops.gated_group_norm(o, g, torch.ones(d, device=dev), 1e-6, yy, group=d, gate_kind="silu"), flush, reps=reps)
        record(f"gated_head_norm_{tag}", t, bytes_=T * H * d * (4 + 2 + 2))
        ya, yb = torch.randn(T, W, device=dev), torch.randn(T, W, device=dev)
        t = _timed(lambda: ops.branch_norm_sum(y, [(ya, nw), (yb, nw)], 0.5, 1e-6), flush, reps=reps)
        record(f"branch_norm_sum_{tag}", t, bytes_=T * W * 4 * 4)
    return out


def netinex_kernel_numbers(s: dict, peaks: dict) -> dict:
    """The Netinex design's own kernels alone at the layer sizes ``s``, measured as ``kernel_numbers`` measures; the
    experts beside the plain feed-forward of as many weights per token (``bf16``: FLOPs over the measured cuBLAS rate)."""
    import torch
    from types import SimpleNamespace

    from ferrisinfer_b200.engine.workspace import Workspace
    from ferrisinfer_b200.kernels import ops

    dev = torch.device("cuda")
    bf = torch.bfloat16
    flush = torch.zeros(96 << 20, dtype=torch.float32, device=dev)  # 384 MB
    W, H, G, d, ff = s["width"], s["heads"], s["kv_heads"], s["dim"], s["ff"]
    hbm = peaks["hbm_gbs"] * 1e9
    tensor = peaks["bf16_tflops"] * 1e12
    ws = Workspace(dev)
    out = {}

    def ctx_of(q_lens, start):
        S = len(q_lens)
        q_start = [0]
        for n in q_lens:
            q_start.append(q_start[-1] + n)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        return SimpleNamespace(num_tokens=q_start[-1], num_seqs=S, max_q_len=max(q_lens), workspace=ws,
                               max_kv_len=start + max(q_lens),
                               token_seq=i32([i for i in range(S) for _ in range(q_lens[i])]),
                               positions=i32([start + j for i in range(S) for j in range(q_lens[i])]),
                               seq_q_start=i32(q_start), seq_start_pos=i32([start] * S), seq_state_slot=i32(list(range(S))))

    def record(name, seconds, bytes_=None, flops=None, tensor_flops=None):
        e = {"us": round(seconds * 1e6, 1)}
        if bytes_ is not None:
            e["GBps"] = round(bytes_ / seconds / 1e9, 1)
            e["frac_hbm"] = round(bytes_ / seconds / hbm, 3)
        if flops is not None:
            e["TFLOPs_fp32"] = round(flops / seconds / 1e12, 2)
            e["frac_fp32_nominal"] = round(flops / seconds / (FP32_NOMINAL_TFLOPS * 1e12), 3)
        if tensor_flops is not None:
            e["TFLOPs_bf16"] = round(tensor_flops / seconds / 1e12, 1)
            e["frac_bf16_measured"] = round(tensor_flops / seconds / tensor, 3)
        out[name] = e

    # ---- retention: the decayed linear attention with q and k rotated and k scaled on the way in
    freq = torch.exp(-math.log(1e6) * torch.arange(d // 2, device=dev, dtype=torch.float32) * 2 / d)
    table = ops.RotaryTable(freq, d, interleaved=False)
    for name, q_lens in (("retention_decode_b64", [1] * 64), ("retention_prefill_2048", [2048])):
        T, S = sum(q_lens), len(q_lens)
        proj = torch.randn(T, 4 * H * d, device=dev).to(bf)
        state = torch.zeros(S + 1, H, d, d, device=dev)
        o = torch.empty(T, H * d, device=dev)
        decay = torch.full((H,), 0.97, device=dev)
        ctx = ctx_of(q_lens, 7)
        t = _timed(lambda: ops.linear_attention(proj, (0, H * d, 2 * H * d), o, state, decay, ctx, H, d, d, silu=False,
                                                rotary=table, k_scale=d ** -0.5), flush)
        moved = 2 * S * H * d * d * 4 + T * 3 * H * d * 2 + T * H * d * 4
        record(name, t, bytes_=moved, flops=4.0 * T * H * d * d)
    # ---- attention within chunks, the values read from the raw keys' rows; and the kernel ahead of it
    itab = ops.RotaryTable(freq, d, interleaved=True, magnitude=1.1)
    for name, batch, q_len, ctx_len in (("decode_b64", 64, 1, 2047), ("prefill_2048", 1, 2048, 0)):
        T = batch * q_len
        pages_each = (ctx_len + q_len + 15) // 16
        k = torch.randn(batch * pages_each + 1, G, 16, d, device=dev).to(bf)
        v = torch.randn_like(k)
        tables = torch.arange(batch * pages_each, dtype=torch.int32, device=dev).view(batch, pages_each)
        qk = torch.randn(T, (H + G) * d, device=dev).to(bf)
        o = torch.empty(T, H * d, dtype=bf, device=dev)
        ctx = ctx_of([q_len] * batch, ctx_len)
        t = _timed(lambda: ops.paged_attention_simt(qk, o, k, v, tables, ctx.token_seq, ctx.positions, H, G, d, 0,
                                                    1.0 / math.sqrt(d), v_head_dim=d, max_q_len=q_len,
                                                    max_kv_len=ctx_len + q_len, workspace=ws, chunk=WINDOW), flush)
        keys = sum((ctx_len + j) % WINDOW + 1 for j in range(q_len)) * batch
        record(f"chunk_attention_{name}", t, flops=4.0 * keys * H * d,
               bytes_=batch * G * (ctx_len % WINDOW + 1) * 2 * d * 2 + T * H * d * 4 if q_len == 1 else None)
        slots = (tables[ctx.token_seq.long(), (ctx.positions // 16).long()] * 16 + ctx.positions % 16).int()
        qn, kn = torch.ones(H * d, device=dev), torch.ones(G * d, device=dev)
        t = _timed(lambda: ops.qk_norm_rotary_cache_write(qk, ctx, slots, k, v, H, G, d, d, qn, kn, 1e-6, itab,
                                                          values_from_keys=True), flush, reps=10)
        record(f"qk_norm_rotary_{name}", t, bytes_=T * (2 * H * d + 3 * G * d) * 2)
    # ---- row-wise kernels of a long step and of a decode step
    for tag, T in (("2048", 2048), ("b64", 64)):
        reps = 10 if T <= 64 else 1
        h = torch.randn(T, W, device=dev)
        w1, b1, alpha = torch.ones(W, device=dev), torch.zeros(W, device=dev), torch.full((1,), 0.7, device=dev)
        a = torch.empty(T, W, dtype=bf, device=dev)
        t = _timed(lambda: ops.dynamic_tanh(h, w1, b1, alpha, a), flush, reps=reps)
        record(f"dynamic_tanh_{tag}", t, bytes_=T * W * (4 + 2))
        o = torch.randn(T, H * d, device=dev)
        g = torch.randn(T, H * d, device=dev).to(bf)
        y = torch.empty(T, H * d, dtype=bf, device=dev)
        one = torch.ones(1, device=dev)
        t = _timed(lambda: ops.gated_group_norm(o, g, one, 1e-6, y, group=d, gate_kind="silu"), flush, reps=reps)
        record(f"head_norm_silu_gate_{tag}", t, bytes_=T * H * d * (4 + 2 + 2))
        logits = torch.randn(T, VOCAB, device=dev)
        t = _timed(lambda: ops.softcap_(logits, 30.0), flush, reps=reps)
        record(f"softcap_{tag}", t, bytes_=T * VOCAB * 8)
    # ---- the experts beside the plain feed-forward of as many weights per token
    eff = netinex_expert_ff(s)
    gate_up = (torch.randn(EXPERTS, 2 * eff, W, device=dev) / math.sqrt(W)).to(bf)
    down = (torch.randn(EXPERTS, W, eff, device=dev) / math.sqrt(eff)).to(bf)
    router = torch.randn(EXPERTS, W, device=dev).to(bf)
    rb = torch.zeros(EXPERTS, device=dev)
    w_up = (torch.randn(ff, W, device=dev) / math.sqrt(W)).to(bf)
    w_down = (torch.randn(W, ff, device=dev) / math.sqrt(ff)).to(bf)
    for tag, T in (("b8", 8), ("b64", 64), ("2048", 2048)):
        x = torch.randn(T, W, device=dev).to(bf)
        hrow = torch.zeros(T, W, device=dev)
        ids = torch.empty(T, TOP, dtype=torch.int32, device=dev)
        wts = torch.empty(T, TOP, device=dev)
        t = _timed(lambda: ops.moe_router(x, router, rb, ids, wts, TOP), flush, reps=10)
        record(f"router_{tag}", t, bytes_=T * W * 2 + EXPERTS * W * 2)
        distinct = int(torch.unique(ids).numel())
        t = _timed(lambda: ops.moe_experts(x, gate_up, down, ids, wts, hrow, ws, accumulate=True), flush)
        record(f"experts_{tag}", t, bytes_=distinct * 3 * W * eff * 2 + T * W * (2 + 8),
               tensor_flops=2.0 * T * TOP * 3 * W * eff)
        out[f"experts_{tag}"]["distinct_experts"] = distinct
        act = torch.empty(T, ff, dtype=bf, device=dev)

        def dense():
            ops.gemm_activation(x, w_up, act, "silu")
            ops.gemm(act, w_down, None, hrow, accumulate=True)

        t = _timed(dense, flush)
        record(f"dense_feed_forward_{tag}", t, bytes_=2 * W * ff * 2 + T * W * (2 + 8), tensor_flops=2.0 * T * 2 * W * ff)
    return out


def sumevik_kernel_numbers(s: dict, peaks: dict) -> dict:
    """The Sumevik design's own kernels alone at the layer sizes ``s``, measured as ``kernel_numbers`` measures; its gated
    products beside the SiLU-gated ones, its router and experts beside the Netinex design's."""
    import torch
    from types import SimpleNamespace

    from ferrisinfer_b200.engine.workspace import Workspace
    from ferrisinfer_b200.kernels import ops

    dev = torch.device("cuda")
    bf = torch.bfloat16
    flush = torch.zeros(96 << 20, dtype=torch.float32, device=dev)  # 384 MB
    W, H, G, d, ff = s["width"], s["heads"], s["kv_heads"], s["dim"], s["ff"]
    hbm = peaks["hbm_gbs"] * 1e9
    tensor = peaks["bf16_tflops"] * 1e12
    ws = Workspace(dev)
    out = {}

    def ctx_of(q_lens, start):
        S = len(q_lens)
        q_start = [0]
        for n in q_lens:
            q_start.append(q_start[-1] + n)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        return SimpleNamespace(num_tokens=q_start[-1], num_seqs=S, max_q_len=max(q_lens), workspace=ws,
                               max_kv_len=start + max(q_lens),
                               token_seq=i32([i for i in range(S) for _ in range(q_lens[i])]),
                               positions=i32([start + j for i in range(S) for j in range(q_lens[i])]),
                               seq_q_start=i32(q_start), seq_start_pos=i32([start] * S), seq_state_slot=i32(list(range(S))))

    def record(name, seconds, bytes_=None, flops=None, tensor_flops=None):
        e = {"us": round(seconds * 1e6, 1)}
        if bytes_ is not None:
            e["GBps"] = round(bytes_ / seconds / 1e9, 1)
            e["frac_hbm"] = round(bytes_ / seconds / hbm, 3)
        if flops is not None:
            e["TFLOPs_fp32"] = round(flops / seconds / 1e12, 2)
            e["frac_fp32_nominal"] = round(flops / seconds / (FP32_NOMINAL_TFLOPS * 1e12), 3)
        if tensor_flops is not None:
            e["TFLOPs_bf16"] = round(tensor_flops / seconds / 1e12, 1)
            e["frac_bf16_measured"] = round(tensor_flops / seconds / tensor, 3)
        out[name] = e

    # ---- the recurrent unit: gates (block-diagonal products, sigmoids, decay) and the scan over channels
    C, blocks = W, H
    bs = C // blocks
    wa = (torch.randn(blocks, bs, bs, device=dev) / math.sqrt(bs)).to(bf)
    wi = (torch.randn(blocks, bs, bs, device=dev) / math.sqrt(bs)).to(bf)
    ba, bi, rate = torch.zeros(C, device=dev), torch.zeros(C, device=dev), torch.full((C,), 0.05, device=dev)
    for tag, q_lens in (("decode_b64", [1] * 64), ("prefill_2048", [2048])):
        T, S = sum(q_lens), len(q_lens)
        reps = 10 if T <= 64 else 1
        u = torch.randn(T, C, device=dev).to(bf)
        ybranch = torch.randn(T, C, device=dev).to(bf)
        a, b = torch.empty(T, C, device=dev), torch.empty(T, C, device=dev)
        y = torch.empty(T, C, dtype=bf, device=dev)
        state = torch.zeros(S + 1, C, device=dev)
        ctx = ctx_of(q_lens, 5)
        t = _timed(lambda: ops.rglru_gates(u, wa, wi, ba, bi, rate, a, b, 8.0), flush, reps=reps)
        record(f"recurrent_gates_{tag}", t, bytes_=2 * C * bs * 2 + T * C * (2 + 8), flops=2.0 * T * 2 * C * bs)
        if T >= ops.RGLRU_TENSOR_CORE_MIN_TOKENS:  # the form a long bf16 step takes: the products on the tensor cores
            stored = (wa.transpose(1, 2).contiguous(), wi.transpose(1, 2).contiguous())
            t = _timed(lambda: ops.rglru_gates(u, wa, wi, ba, bi, rate, a, b, 8.0, stored=stored), flush, reps=reps)
            record(f"recurrent_gates_tensor_cores_{tag}", t, bytes_=2 * C * bs * 2 + T * C * (2 + 8),
                   tensor_flops=2.0 * T * 2 * C * bs)
        a.uniform_(-0.5, 0.0)  # (in case the gates left something else: the scan takes logarithms of decays)
        t = _timed(lambda: ops.rglru_scan(a, b, ybranch, y, state, ctx), flush, reps=reps)
        record(f"recurrent_scan_{tag}", t, bytes_=T * C * (8 + 2 + 2) + 2 * S * C * 4)
        cw = torch.randn(C, 4, device=dev) * 0.1
        cb = torch.zeros(C, device=dev)
        hist = torch.zeros(S + 1, 3, C, device=dev)
        wide = torch.randn(T, 2 * C, device=dev).to(bf)
        t = _timed(lambda: ops.short_conv(wide[:, C:], u, cw, hist, ctx, bias=cb, residual=False), flush, reps=reps)
        record(f"recurrent_conv_{tag}", t, bytes_=T * C * 4 + (S * 3 * C * 8 if T <= 64 else 0))
    # ---- the gated linear attention: the recurrence with a decay per key channel, and the norm per head with its gate
    dk = d // 2
    for tag, q_lens in (("decode_b64", [1] * 64), ("prefill_2048", [2048])):
        T, S = sum(q_lens), len(q_lens)
        proj = (torch.randn(T, 2 * H * dk + 2 * H * d, device=dev) / 4.0).to(bf)
        z = 3.0 + torch.randn(T, H * dk, device=dev)
        state = torch.zeros(S + 1, H, d, dk, device=dev)
        o = torch.empty(T, H * d, device=dev)
        ctx = ctx_of(q_lens, 0)
        t = _timed(lambda: ops.row_decay_recurrence(proj[:, :H * dk], proj[:, H * dk:2 * H * dk], proj[:, 2 * H * dk:2 * H * dk + H * d],
                                                    z, 1.0 / 8.0, o, state, ctx, H, dk, d, q_scale=dk ** -0.5), flush)
        moved = 2 * S * H * dk * d * 4 + T * (2 * H * dk + H * d) * 2 + T * H * dk * 4 + T * H * d * 4
        record(f"linear_attention_row_decay_{tag}", t, bytes_=moved, flops=4.0 * T * H * dk * d)
    # ---- the attention's own kernels: norm per head + rotation + cache write, the chunked attention with value heads of
    # their own, the gate on its output
    freq = torch.exp(-math.log(1e6) * torch.arange(d // 4, device=dev, dtype=torch.float32) * 4 / d)
    itab = ops.RotaryTable(freq, d // 2, interleaved=True, freq_lo=torch.zeros_like(freq))
    for name, batch, q_len, ctx_len in (("decode_b64", 64, 1, 2047), ("prefill_2048", 1, 2048, 0)):
        T = batch * q_len
        reps = 10 if T <= 64 else 1
        pages_each = (ctx_len + q_len + 15) // 16
        k = torch.randn(batch * pages_each + 1, G, 16, d, device=dev).to(bf)
        v = torch.randn_like(k)
        tables = torch.arange(batch * pages_each, dtype=torch.int32, device=dev).view(batch, pages_each)
        rows = torch.randn(T, (H + 2 * G) * d + H * d, device=dev).to(bf)  # q, k, v and the gate's columns
        qkv, gate = rows[:, :(H + 2 * G) * d], rows[:, (H + 2 * G) * d:]
        o = torch.empty(T, H * d, dtype=bf, device=dev)
        ctx = ctx_of([q_len] * batch, ctx_len)
        slots = (tables[ctx.token_seq.long(), (ctx.positions // 16).long()] * 16 + ctx.positions % 16).int()
        qn, kn = torch.ones(d, device=dev), torch.ones(d, device=dev)
        t = _timed(lambda: ops.qk_norm_rotary_cache_write(qkv, ctx, slots, k, v, H, G, d, d, qn, kn, 1e-6, itab, per_head=True),
                   flush, reps=10)
        record(f"head_norm_rotary_{name}", t, bytes_=T * (2 * H * d + 4 * G * d) * 2)
        t = _timed(lambda: ops.paged_attention_simt(qkv, o, k, v, tables, ctx.token_seq, ctx.positions, H, G, d, 0,
                                                    1.0 / math.sqrt(d), v_head_dim=d, max_q_len=q_len,
                                                    max_kv_len=ctx_len + q_len, workspace=ws, chunk=WINDOW), flush)
        keys = sum((ctx_len + j) % WINDOW + 1 for j in range(q_len)) * batch
        record(f"chunk_attention_{name}", t, flops=4.0 * keys * H * d,
               bytes_=batch * G * (ctx_len % WINDOW + 1) * 2 * d * 2 + T * H * d * 4 if q_len == 1 else None)
        t = _timed(lambda: ops.gate_mul(o, gate, o, "sigmoid", 0.9), flush, reps=reps)
        record(f"output_gate_{name}", t, bytes_=T * H * d * 6)
        og = torch.randn(T, H * d, device=dev)
        yy = torch.empty(T, H * d, dtype=bf, device=dev)
        t = _timed(lambda: ops.gated_group_norm(og, gate, torch.ones(d, device=dev), 1e-6, yy, group=d, gate_kind="silu"), flush, reps=reps)
        record(f"head_norm_silu_gate_{name}", t, bytes_=T * H * d * (4 + 2 + 2))
    # ---- the gated feed-forward: the tanh GELU in the products' epilogues beside the SiLU of the other designs
    inter = sumevik_dense_ff(s)
    gate_up_w = (torch.randn(2 * inter, W, device=dev) / math.sqrt(W)).to(bf)
    for tag, T in (("b8", 8), ("b64", 64), ("2048", 2048)):
        x = torch.randn(T, W, device=dev).to(bf)
        act = torch.empty(T, inter, dtype=bf, device=dev)
        for kind in ("gelu_tanh", "silu"):
            t = _timed(lambda: ops.gemm_gated(x, gate_up_w, act, kind, 0.0, ws), flush)
            record(f"gated_product_{kind}_{tag}", t, bytes_=2 * inter * W * 2 + T * (W + inter) * 2,
                   tensor_flops=2.0 * T * 2 * inter * W)
    # ---- the scored router and the experts with a clamped gate and identity experts
    eff = netinex_expert_ff(s)
    outputs = EXPERTS + SUMEVIK_IDENTITY
    gate_up = (torch.randn(EXPERTS, 2 * eff, W, device=dev) / math.sqrt(W)).to(bf)
    down = (torch.randn(EXPERTS, W, eff, device=dev) / math.sqrt(eff)).to(bf)
    router = torch.randn(outputs, W, device=dev).to(bf)
    corr = torch.zeros(outputs, device=dev)
    for tag, T in (("b8", 8), ("b64", 64), ("2048", 2048)):
        x = torch.randn(T, W, device=dev).to(bf)
        hrow = torch.zeros(T, W, device=dev)
        ids = torch.empty(T, TOP, dtype=torch.int32, device=dev)
        wts = torch.empty(T, TOP, device=dev)
        idw = torch.empty(T, device=dev)
        scored = {"correction": corr, "groups": 2, "keep": 1, "with_weights": EXPERTS, "identity_w": idw}
        t = _timed(lambda: ops.moe_router(x, router, None, ids, wts, TOP, scored=scored), flush, reps=10)
        record(f"scored_router_{tag}", t, bytes_=T * W * 2 + outputs * W * 2)
        chosen = torch.unique(ids)
        distinct = int((chosen < EXPERTS).sum())
        pairs = int((ids < EXPERTS).sum())
        t = _timed(lambda: ops.moe_experts(x, gate_up, down, ids, wts, hrow, ws, accumulate=True, activation="clamped_swish",
                                           limit=7.0, identity_w=idw), flush)
        record(f"experts_clamped_{tag}", t, bytes_=distinct * 3 * W * eff * 2 + T * W * (2 + 8),
               tensor_flops=2.0 * pairs * 3 * W * eff)
        out[f"experts_clamped_{tag}"]["distinct_experts"] = distinct
        out[f"experts_clamped_{tag}"]["pairs_with_weights"] = pairs
    return out


def retezen_kernel_numbers(s: dict, peaks: dict) -> dict:
    """The Retezen design's own kernels alone at the layer sizes ``s``, measured as ``kernel_numbers`` measures; the attention
    beside the same kernel without blocks, the clamped gate beside the SiLU one, experts whose weights go onto their inputs."""
    import torch
    from types import SimpleNamespace

    from ferrisinfer_b200.engine.workspace import Workspace
    from ferrisinfer_b200.kernels import ops

    dev = torch.device("cuda")
    bf = torch.bfloat16
    flush = torch.zeros(96 << 20, dtype=torch.float32, device=dev)  # 384 MB
    W, H, G, d = s["width"], s["heads"], s["kv_heads"], s["dim"]
    hbm = peaks["hbm_gbs"] * 1e9
    tensor = peaks["bf16_tflops"] * 1e12
    ws = Workspace(dev)
    out = {}

    def ctx_of(q_lens, start):
        S = len(q_lens)
        q_start = [0]
        for n in q_lens:
            q_start.append(q_start[-1] + n)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        return SimpleNamespace(num_tokens=q_start[-1], num_seqs=S, max_q_len=max(q_lens), workspace=ws,
                               max_kv_len=start + max(q_lens),
                               token_seq=i32([i for i in range(S) for _ in range(q_lens[i])]),
                               positions=i32([start + j for i in range(S) for j in range(q_lens[i])]),
                               seq_q_start=i32(q_start), seq_start_pos=i32([start] * S), seq_state_slot=i32(list(range(S))))

    def record(name, seconds, bytes_=None, flops=None, tensor_flops=None):
        e = {"us": round(seconds * 1e6, 1)}
        if bytes_ is not None:
            e["GBps"] = round(bytes_ / seconds / 1e9, 1)
            e["frac_hbm"] = round(bytes_ / seconds / hbm, 3)
        if flops is not None:
            e["TFLOPs_fp32"] = round(flops / seconds / 1e12, 2)
            e["frac_fp32_nominal"] = round(flops / seconds / (FP32_NOMINAL_TFLOPS * 1e12), 3)
        if tensor_flops is not None:
            e["TFLOPs_bf16"] = round(tensor_flops / seconds / 1e12, 1)
            e["frac_bf16_measured"] = round(tensor_flops / seconds / tensor, 3)
        out[name] = e

    # ---- the attention over a window and blocks, beside the same kernel over the window alone, and what stands ahead of it
    P = RETEZEN_POOL
    for name, batch, q_len, ctx_len in (("decode_b64", 64, 1, 2047), ("decode_b8", 8, 1, 2047), ("prefill_2048", 1, 2048, 0)):
        T = batch * q_len
        reps = 10 if T <= 64 else 1
        pages_each = (ctx_len + q_len + 15) // 16
        runs_each = (pages_each + P - 1) // P
        k = torch.randn(batch * pages_each + 1, G, 16, d, device=dev).to(bf)
        v = torch.randn_like(k)
        pk = torch.randn(batch * runs_each + 1, G, 16, d, device=dev).to(bf)
        tables = torch.arange(batch * pages_each, dtype=torch.int32, device=dev).view(batch, pages_each)
        ptables = torch.arange(batch * runs_each, dtype=torch.int32, device=dev).view(batch, runs_each)
        pooled = ops.PooledKeys(pk, torch.randn_like(pk), ptables, P)
        qkv = torch.randn(T, (H + 2 * G) * d, device=dev).to(bf)
        o = torch.empty(T, H * d, dtype=bf, device=dev)
        ctx = ctx_of([q_len] * batch, ctx_len)
        window = [min(WINDOW, ctx_len + j + 1) for j in range(q_len)]
        blocks = [max(0, ctx_len + j + 1 - WINDOW) // P for j in range(q_len)]
        for what, pool_arg, keys in (("pooled_attention", pooled, sum(window) + sum(blocks)), ("window_attention", None, sum(window))):
            t = _timed(lambda: ops.paged_attention_simt(qkv, o, k, v, tables, ctx.token_seq, ctx.positions, H, G, d, WINDOW,
                                                        1.0 / math.sqrt(d), v_head_dim=d, max_q_len=q_len,
                                                        max_kv_len=ctx_len + q_len, workspace=ws, pooled=pool_arg), flush)
            record(f"{what}_{name}", t, flops=4.0 * keys * batch * H * d,
                   bytes_=batch * G * keys * 2 * d * 2 + T * H * d * 4 if q_len == 1 else None)
        slots = (tables[ctx.token_seq.long(), (ctx.positions // 16).long()] * 16 + ctx.positions % 16).int()
        row = (ctx.positions // P).long()
        pslots = (ptables[ctx.token_seq.long(), row // 16] * 16 + row % 16).int()
        pslots = torch.where((ctx.positions + 1) % P == 0, pslots, torch.full_like(pslots, -1))
        qn, kn, lam = torch.ones(H * d, device=dev), torch.ones(G * d, device=dev), torch.full((1,), 0.3, device=dev)
        first = torch.randn(T, G * d, device=dev).to(bf)
        extra = {}
        if q_len == 1:  # (position 2,047 completes a block: the means are in this number)
            extra = dict(pooled=pooled, pool_slots=pslots, block_tables=tables)
        t = _timed(lambda: ops.qk_norm_rotary_cache_write(qkv, ctx, slots, k, v, H, G, d, d, qn, kn, 1e-6, None,
                                                          mixed_values=first, mix_lambda=lam, **extra), flush, reps=10)
        record(f"qk_norm_mix_{name}", t, bytes_=T * (2 * H * d + 4 * G * d + G * d) * 2 + (batch * (P + 1) * 2 * G * d * 2 if extra else 0))
        if q_len > 1:
            t = _timed(lambda: ops.pool_blocks(k, v, pooled, pslots, tables, ctx), flush, reps=10)
            record(f"block_means_{name}", t, bytes_=(T // P) * (P + 1) * 2 * G * d * 2)
    # ---- row-wise kernels of a long step and of a decode step
    for tag, T in (("2048", 2048), ("b64", 64), ("b8", 8)):
        reps = 10 if T <= 64 else 1
        y, h, nw = torch.randn(T, W, device=dev), torch.zeros(T, W, device=dev), torch.ones(W, device=dev)
        rows = torch.empty(T, W, dtype=bf, device=dev)
        t = _timed(lambda: ops.rmsnorm_add(y, nw, 1e-6, h, rows), flush, reps=reps)
        record(f"norm_add_{tag}", t, bytes_=T * W * (4 + 4 + 4 + 2))
        table, pos = torch.randn(VOCAB, W, device=dev).to(bf), torch.randn(4096, W, device=dev).to(bf)
        ids = torch.randint(0, VOCAB, (T,), dtype=torch.int32, device=dev)
        ps = torch.arange(T, dtype=torch.int32, device=dev)
        t = _timed(lambda: ops.embed_positions(table, pos, ids, ps, h, rows), flush, reps=reps)
        record(f"embed_positions_{tag}", t, bytes_=T * W * (2 + 2 + 4 + 2))
    # ---- the gated feed-forward: the clamped gate in the products' epilogues beside the SiLU one
    inter = sumevik_dense_ff(s)
    gate_up_w = (torch.randn(2 * inter, W, device=dev) / math.sqrt(W)).to(bf)
    for tag, T in (("b8", 8), ("b64", 64), ("2048", 2048)):
        x = torch.randn(T, W, device=dev).to(bf)
        act = torch.empty(T, inter, dtype=bf, device=dev)
        for kind in ("clamped_swish", "silu"):
            t = _timed(lambda: ops.gemm_gated(x, gate_up_w, act, kind, 7.0, ws), flush)
            record(f"gated_product_{kind}_{tag}", t, bytes_=2 * inter * W * 2 + T * (W + inter) * 2,
                   tensor_flops=2.0 * T * 2 * inter * W)
    # ---- the sigmoid router and the experts with weights on their inputs
    eff = netinex_expert_ff(s)
    gate_up = (torch.randn(EXPERTS, 2 * eff, W, device=dev) / math.sqrt(W)).to(bf)
    down = (torch.randn(EXPERTS, W, eff, device=dev) / math.sqrt(eff)).to(bf)
    router = torch.randn(EXPERTS, W, device=dev).to(bf)
    for tag, T in (("b8", 8), ("b64", 64), ("2048", 2048)):
        x = torch.randn(T, W, device=dev).to(bf)
        hrow = torch.zeros(T, W, device=dev)
        ids = torch.empty(T, TOP, dtype=torch.int32, device=dev)
        wts = torch.empty(T, TOP, device=dev)
        t = _timed(lambda: ops.moe_router(x, router, None, ids, wts, TOP, sigmoid=True), flush, reps=10)
        record(f"sigmoid_router_{tag}", t, bytes_=T * W * 2 + EXPERTS * W * 2)
        distinct = int(torch.unique(ids).numel())
        t = _timed(lambda: ops.moe_experts(x, gate_up, down, ids, wts, hrow, ws, accumulate=False, input_weights=True), flush)
        record(f"experts_input_weights_{tag}", t, bytes_=distinct * 3 * W * eff * 2 + T * W * (2 + 4),
               tensor_flops=2.0 * T * TOP * 3 * W * eff)
        out[f"experts_input_weights_{tag}"]["distinct_experts"] = distinct
    return out


def lukelorn_kernel_numbers(s: dict, peaks: dict) -> dict:
    """The Lukelorn design's own kernels alone at the layer sizes ``s``, measured as ``kernel_numbers`` measures (prompt portions
    four launches back to back: a form of two launches would else be timed together with the host's way to both), each beside the
    like kernel of the designs that were there before (the delta rule with a decay per head, attention over a window alone, over
    a latent without one, experts with a gate of as many weights)."""
    import torch
    from types import SimpleNamespace

    from ferrisinfer_b200.engine.workspace import Workspace
    from ferrisinfer_b200.kernels import ops
    from ferrisinfer_b200.parts.position import ScaledRotary

    dev = torch.device("cuda")
    bf = torch.bfloat16
    flush = torch.zeros(96 << 20, dtype=torch.float32, device=dev)  # 384 MB
    W, H, G, d = s["width"], s["heads"], s["kv_heads"], s["dim"]
    hbm, tensor = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    ws = Workspace(dev)
    out = {}

    def ctx_of(q_lens, start):
        S = len(q_lens)
        q_start = [0]
        for n in q_lens:
            q_start.append(q_start[-1] + n)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        return SimpleNamespace(num_tokens=q_start[-1], num_seqs=S, max_q_len=max(q_lens), workspace=ws,
                               max_kv_len=start + max(q_lens),
                               token_seq=i32([i for i in range(S) for _ in range(q_lens[i])]),
                               positions=i32([start + j for i in range(S) for j in range(q_lens[i])]),
                               seq_q_start=i32(q_start), seq_start_pos=i32([start] * S), seq_state_slot=i32(list(range(S))))

    def record(name, seconds, bytes_=None, flops=None, tensor_flops=None):
        e = {"us": round(seconds * 1e6, 1)}
        if bytes_ is not None:
            e["GBps"] = round(bytes_ / seconds / 1e9, 1)
            e["frac_hbm"] = round(bytes_ / seconds / hbm, 3)
        if flops is not None:
            e["TFLOPs_fp32"] = round(flops / seconds / 1e12, 2)
            e["frac_fp32_nominal"] = round(flops / seconds / (FP32_NOMINAL_TFLOPS * 1e12), 3)
        if tensor_flops is not None:
            e["TFLOPs_bf16"] = round(tensor_flops / seconds / 1e12, 1)
            e["frac_bf16_measured"] = round(tensor_flops / seconds / tensor, 3)
        out[name] = e

    rank, rot, qr = 192, 64, lukelorn_q_rank(s)
    randn = lambda *shape: torch.randn(*shape, device=dev)
    for name, batch, q_len, ctx_len in (("decode_b64", 64, 1, 2047), ("decode_b8", 8, 1, 2047), ("prefill_2048", 1, 2048, 0)):
        T = batch * q_len
        reps = 10 if T <= 64 else 4
        pages_each = (ctx_len + q_len + 15) // 16
        tables = torch.arange(batch * pages_each, dtype=torch.int32, device=dev).view(batch, pages_each)
        ctx = ctx_of([q_len] * batch, ctx_len)
        slots = (tables[ctx.token_seq.long(), (ctx.positions // 16).long()] * 16 + ctx.positions % 16).int()
        # ---- attention: a window with kept tokens, a soft cap, a sink and gates, beside the window alone
        k = randn(batch * pages_each + 1, G, 16, d).to(bf)
        v = torch.randn_like(k)
        width = (H + 2 * G) * d + H
        qkv = randn(T, (width + 7) // 8 * 8).to(bf)
        o = torch.empty(T, H * d, dtype=bf, device=dev)
        terms = ops.ScoreTerms(sink=torch.zeros(H, device=dev), softcap=50.0, gate=qkv[:, (H + 2 * G) * d:width])
        seen = [min(WINDOW, ctx_len + j + 1) for j in range(q_len)]
        kept = [min(LUKELORN_KEEP, max(0, ctx_len + j + 1 - WINDOW)) for j in range(q_len)]
        for what, keep, t_, keys in (("kept_capped_attention", LUKELORN_KEEP, terms, sum(seen) + sum(kept)),
                                     ("window_attention", 0, None, sum(seen))):
            t = _timed(lambda: ops.paged_attention_simt(qkv, o, k, v, tables, ctx.token_seq, ctx.positions, H, G, d, WINDOW,
                                                        1.0 / math.sqrt(d), score_slopes=t_, v_head_dim=d, max_q_len=q_len,
                                                        max_kv_len=ctx_len + q_len, workspace=ws, keep_first=keep), flush, reps=reps)
            record(f"{what}_{name}", t, flops=4.0 * keys * batch * H * d,
                   bytes_=batch * G * keys * 2 * d * 2 + T * H * d * 4 if q_len == 1 else None)
        table = ScaledRotary(d, 5e5, "interleaved", {"kind": "wavelength", "factor": 4.0, "low": 1.0, "high": 4.0, "original": 2048}).table(dev)
        rows = qkv[:, :(H + 2 * G) * d]
        t = _timed(lambda: ops.qk_norm_rotary_cache_write(rows, ctx, slots, k, v, H, G, d, d, None, None, 0.0, table), flush, reps=10)
        record(f"rotary_cache_write_{name}", t, bytes_=T * (2 * H * d + 4 * G * d) * 2)
        # ---- attention over the latent, in a window and over every key
        kl = randn(batch * pages_each + 1, 1, 16, rank + rot).to(bf)
        ql = randn(T, H * (rank + rot)).to(bf)
        ol = torch.empty(T, H * rank, dtype=bf, device=dev)
        for what, window in (("latent_window_attention", WINDOW), ("latent_attention", 0)):
            keys = (sum(seen) if window else sum(ctx_len + j + 1 for j in range(q_len))) * batch
            t = _timed(lambda: ops.paged_attention_simt(ql, ol, kl, None, tables, ctx.token_seq, ctx.positions, H, 1, rank + rot,
                                                        window, 0.07, v_head_dim=rank, max_q_len=q_len, max_kv_len=ctx_len + q_len,
                                                        workspace=ws, values_in_keys=True), flush, reps=reps)
            record(f"{what}_{name}", t, flops=2.0 * keys * H * (2 * rank + rot),
                   bytes_=keys * (rank + rot) * 2 + T * H * (2 * rank + rot) * 2 if q_len == 1 else None)
        lrot = ScaledRotary(rot, 1e6, "interleaved").table(dev)
        proj = randn(T, qr + rank + rot + H).to(bf)
        q = randn(T, H * (d + rot)).to(bf)
        nq, nc = torch.ones(qr, device=dev), torch.ones(rank, device=dev)
        cq = torch.empty(T, qr, dtype=bf, device=dev)
        t = _timed(lambda: ops.latent_prepare(ctx.positions, lrot, 1e-6, H, d, rot, rank, keys=(proj[:, qr:qr + rank + rot], nc, slots, kl),
                                              q_latent=(proj[:, :qr], nq, cq)), flush, reps=10)
        record(f"latent_norms_cache_write_{name}", t, bytes_=T * (2 * qr + 2 * (rank + rot)) * 2)
        t = _timed(lambda: ops.latent_prepare(ctx.positions, lrot, 1e-6, H, d, rot, rank, queries=(q, ql)), flush, reps=10)
        record(f"latent_query_rotation_{name}", t, bytes_=T * 2 * H * rot * 2)
        uk = (randn(H, d, rank) / math.sqrt(d)).to(bf)
        t = _timed(lambda: ops.head_gemm(q, d + rot, uk, ql, rank + rot), flush, reps=reps)
        record(f"head_product_{name}", t, tensor_flops=2.0 * T * H * d * rank, bytes_=H * d * rank * 2 + T * H * (d + rank) * 2)
        # ---- the recurrence: decays per channel beside a decay per head, and what stands around it
        S = batch
        kq, kk = (randn(T, G * d) / math.sqrt(d)).to(bf), (randn(T, G * d) / math.sqrt(d)).to(bf)
        vv, beta = randn(T, H * d).to(bf), torch.full((T, H), 0.5, device=dev)
        z, rates, decay = randn(T, H * d) - 3.0, torch.ones(H, device=dev), torch.full((T, H), 0.97, device=dev)
        state, og = torch.zeros(S + 1, H, d, d, device=dev), torch.empty(T, H * d, device=dev)
        moved = 2 * S * H * d * d * 4 + T * (2 * G * d + H * d) * 2 + T * H * d * 4
        t = _timed(lambda: ops.gated_recurrence(kq, kk, vv, None, beta, og, state, ctx, H, G, d, d, delta_rule=True,
                                                row_decay=(z, rates)), flush, reps=reps)
        record(f"channel_delta_{name}", t, bytes_=moved + T * H * d * 4, flops=7.0 * T * H * d * d)
        if q_len > 1:
            t = _timed(lambda: ops.gated_recurrence(kq, kk, vv, None, beta, og, state, ctx, H, G, d, d, delta_rule=True,
                                                    row_decay=(z, rates), chunks=False), flush, reps=reps)
            record(f"channel_delta_token_by_token_{name}", t, bytes_=moved + T * H * d * 4, flops=7.0 * T * H * d * d)
        t = _timed(lambda: ops.gated_recurrence(kq, kk, vv, decay, beta, og, state, ctx, H, G, d, d, delta_rule=True), flush, reps=reps)
        record(f"delta_rule_{name}", t, bytes_=moved, flops=6.0 * T * H * d * d)
        C = (2 * G + H) * d
        wide, conv = randn(T, C + 64).to(bf), torch.empty(T, C, dtype=bf, device=dev)
        cw, cs = randn(C, 4) * 0.1, torch.zeros(S + 1, 3, C, device=dev)
        t = _timed(lambda: ops.short_conv(wide[:, :C], conv, cw, cs, ctx, residual=False, silu=True), flush, reps=reps)
        record(f"conv_silu_{name}", t, bytes_=T * C * 4 + (S * 3 * C * 8 if q_len == 1 else 0))
        a1, a2, dt = randn(T, d).to(bf), (randn(H * d, d) / math.sqrt(d)).to(bf), torch.zeros(H * d, device=dev)
        t = _timed(lambda: ops.gemm(a1, a2, dt, z), flush, reps=reps)
        record(f"decay_product_{name}", t, bytes_=T * (d * 2 + H * d * 4) + H * d * d * 2, tensor_flops=2.0 * T * H * d * d)
        y, gate = torch.empty(T, H * d, dtype=bf, device=dev), randn(T, H * d).to(bf)
        nw = torch.ones(d, device=dev)
        t = _timed(lambda: ops.gated_group_norm(og, gate, nw, 1e-6, y, group=d, gate_kind="sigmoid"), flush, reps=reps)
        record(f"gated_head_norm_{name}", t, bytes_=T * H * d * (4 + 2 + 2))
        qs, ks = torch.empty(T, G, device=dev), torch.empty(T, G, device=dev)
        t = _timed(lambda: ops.recurrence_gates(gate, None, 0, None, None, None, beta, H,
                                                unit_norm=(conv, 0, G * d, G, d, 1e-6, d ** -0.5, qs, ks)), flush, reps=reps)
        record(f"beta_unit_norms_{name}", t, bytes_=T * (2 * G * d * 2 + H * 2 + H * 4 + 2 * G * 4))
    # ---- experts without a gate beside gated ones of as many weights, weights on their inputs
    router = randn(EXPERTS, W).to(bf)
    for tag, T in (("b64", 64), ("b8", 8), ("2048", 2048)):
        x = randn(T, W).to(bf)
        hrow = torch.zeros(T, W, device=dev)
        ids, wts = torch.empty(T, TOP, dtype=torch.int32, device=dev), torch.empty(T, TOP, device=dev)
        t = _timed(lambda: ops.moe_router(x, router, None, ids, wts, TOP, sigmoid=True), flush, reps=10)
        record(f"sigmoid_router_{tag}", t, bytes_=T * W * 2 + EXPERTS * W * 2)
        distinct = int(torch.unique(ids).numel())
        for what, plain, eff in (("experts_plain", True, lukelorn_expert_ff(s)), ("experts_gated", False, netinex_expert_ff(s))):
            n = 2 if plain else 3
            up = (randn(EXPERTS, (n - 1) * eff, W) / math.sqrt(W)).to(bf)
            down = (randn(EXPERTS, W, eff) / math.sqrt(eff)).to(bf)
            t = _timed(lambda: ops.moe_experts(x, up, down, ids, wts, hrow, ws, accumulate=True, input_weights=True, plain=plain,
                                               activation="relu2" if plain else "silu"), flush, reps=2)
            record(f"{what}_{tag}", t, bytes_=distinct * n * W * eff * 2 + T * W * (2 + 8), tensor_flops=2.0 * T * TOP * n * W * eff)
            out[f"{what}_{tag}"]["distinct_experts"] = distinct
    return out


def run(build_engine, time_decode, time_prefill, peaks, steps=32, warmup=4, sizes=("small", "1B-like"), context=2048,
        prompt=2048, batches=(8, 64), kernels_at="1B-like", design="kugilix") -> dict:
    """``build_engine(cfg, batch, context, extra_tokens)``, ``time_decode`` and ``time_prefill`` are bench.py's.
    ``design`` "kugilix": that design beside Qwen2; "nusudra" or "netinex": that design beside both; "sumevik" or "retezen":
    that design beside Netinex and Qwen2; "lukelorn": that design beside Nusudra, Retezen and Qwen2."""
    import torch

    result = {"context": context, "prompt_tokens": prompt, "window": WINDOW, "sizes": {}}
    for name in sizes:
        s = SIZES[name]
        entry = {"layer_sizes": s, "layer_runs": kugilix_runs(s)}
        designs = (("kugilix", kugilix_config(s)), ("qwen2", qwen2_config(s)))
        if design == "nusudra":
            designs = (("nusudra", nusudra_config(s)),) + designs
        if design == "netinex":
            designs = (("netinex", netinex_config(s)),) + designs
        if design in ("sumevik", "retezen"):
            own = sumevik_config(s) if design == "sumevik" else retezen_config(s)
            designs = ((design, own), ("netinex", netinex_config(s)), ("qwen2", qwen2_config(s)))
        if design == "lukelorn":
            designs = ((design, lukelorn_config(s)), ("nusudra", nusudra_config(s)), ("retezen", retezen_config(s)),
                       ("qwen2", qwen2_config(s)))
        for design_name, cfg in designs:
            numbers = {}
            engine = build_engine(cfg, 1, context, extra_tokens=prompt)
            ms = time_prefill(engine, prompt)
            numbers["prefill_tok_s"] = round(prompt / ms * 1e3, 1)
            numbers["prefill_ms"] = round(ms, 3)
            del engine
            torch.cuda.empty_cache()
            for b in batches:
                engine = build_engine(cfg, b, context)
                times, launches = time_decode(engine, b, context, steps, warmup, regions=3)
                ms = statistics.median(times)
                numbers[f"decode_b{b}_tok_s"] = round(b / ms * 1e3, 1)
                numbers[f"decode_b{b}_ms"] = round(ms, 4)
                numbers[f"decode_b{b}_launches_per_step"] = launches // steps
                del engine
                torch.cuda.empty_cache()
            entry[design_name] = numbers
        result["sizes"][name] = entry
    if kernels_at and design == "lukelorn":
        result["kernels_lukelorn"] = {"at": kernels_at, "expert_ff": lukelorn_expert_ff(SIZES[kernels_at]), "experts": EXPERTS,
                                      "top": TOP, "keep_first": LUKELORN_KEEP, **lukelorn_kernel_numbers(SIZES[kernels_at], peaks)}
    elif kernels_at and design == "retezen":
        result["kernels_retezen"] = {"at": kernels_at, "expert_ff": netinex_expert_ff(SIZES[kernels_at]), "experts": EXPERTS,
                                     "top": TOP, "pool": RETEZEN_POOL, **retezen_kernel_numbers(SIZES[kernels_at], peaks)}
        result["kernels_netinex"] = {"at": kernels_at, "expert_ff": netinex_expert_ff(SIZES[kernels_at]),
                                     "experts": EXPERTS, "top": TOP, **netinex_kernel_numbers(SIZES[kernels_at], peaks)}
    elif kernels_at and design == "sumevik":
        result["kernels_sumevik"] = {"at": kernels_at, "expert_ff": netinex_expert_ff(SIZES[kernels_at]), "experts": EXPERTS,
                                     "identity": SUMEVIK_IDENTITY, "top": TOP,
                                     **sumevik_kernel_numbers(SIZES[kernels_at], peaks)}
        result["kernels_netinex"] = {"at": kernels_at, "expert_ff": netinex_expert_ff(SIZES[kernels_at]),
                                     "experts": EXPERTS, "top": TOP, **netinex_kernel_numbers(SIZES[kernels_at], peaks)}
    elif kernels_at:
        result["kernels"] = {"at": kernels_at, **kernel_numbers(SIZES[kernels_at], peaks)}
        if design == "nusudra":
            result["kernels_nusudra"] = {"at": kernels_at, **nusudra_kernel_numbers(SIZES[kernels_at], peaks)}
        if design == "netinex":
            result["kernels_netinex"] = {"at": kernels_at, "expert_ff": netinex_expert_ff(SIZES[kernels_at]),
                                         "experts": EXPERTS, "top": TOP,
                                         **netinex_kernel_numbers(SIZES[kernels_at], peaks)}
    return result
