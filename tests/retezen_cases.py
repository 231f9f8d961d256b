"""Small Retezen configurations and weights for the tests (see ``netinex_cases`` for how rows are compared).

Projections are drawn with a standard deviation of 1 / sqrt(inputs), norm weights around zero (q and k norms around
one), the numbers that mix values between 0.2 and 0.9, router matrices so that the experts' logits spread over a few
units, so that every mechanism moves the logits by far more than a tolerance.  Sequences are drawn token by token so
that no router's choice is a close call anywhere (``safe_sequence``)."""

from __future__ import annotations

import math
import random

import torch

import plain_retezen as plain
from netinex_cases import random_ids, row_errors  # noqa: F401 (shared with the tests)

CLOSE_CALL = 0.1  # of the size of a router's logits


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(heads, kv_heads, dim, vdim, mask, mlp, v_mix=True, scale=None):
    """``mask``: (window, positions to a pooled block), (window, None) or None."""
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "v_mix": v_mix,
             "scale": scale if scale is not None else 2.0 / math.sqrt(dim)}
    if mask is not None:
        mixer["mask"] = {"size": mask[0]}
        if mask[1] is not None:
            mixer["mask"]["pool"] = mask[1]
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def config(layers, width=64, vocab=97, eps=1e-6, logit_scale=0.7, max_positions=640):
    return {"architecture": "Retezen", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps},
            "logit_scale": logit_scale, "layers": layers}


# A: a dense layer and two mixtures, a window of a page and a half, blocks of five positions, two of six experts
CASE_A = config([layer(4, 2, 32, 24, (24, 5), dense(96, 2.0)), layer(4, 2, 32, 24, (24, 5), moe(64, 6, 2)),
                 layer(4, 2, 32, 24, (24, 5), moe(64, 6, 2))])
# B: every layer another mask (none, a window alone, a window with blocks), mixing from the second layer on and left out
# in between, value heads of other shapes with as many values a token, a layer without a feed-forward, three of seven
# experts, a factor of one on the logits, one kv head
CASE_B = config([layer(3, 1, 40, 24, (21, None), dense(72, 0.5), v_mix=False), layer(4, 2, 16, 20, None, None),
                 layer(4, 4, 24, 10, (33, 7), moe(56, 7, 3), scale=0.4), layer(2, 1, 64, 64, (9, 4), moe(40, 5, 1), v_mix=False),
                 layer(8, 1, 32, 40, (18, 11), dense(48, 5.0))], width=48, vocab=131, eps=1e-5, logit_scale=1.0)
# C: head sizes and widths that are no multiple of two, a window of one token, blocks of one position, blocks far longer
# than the window, blocks as long as a page, as many kv heads as heads, all experts chosen
CASE_C = config([layer(3, 3, 15, 9, (1, 3), moe(33, 3, 3)), layer(3, 3, 15, 9, (5, 16), moe(80, 9, 4)),
                 layer(2, 1, 33, 27, (19, 1), dense(50, 1.5)), layer(6, 3, 8, 9, (7, 40), None)], width=43, vocab=61, eps=1e-5,
                logit_scale=-1.3)
# D: window and blocks at page borders exactly, heads of 128, a width that is no multiple of eight, no mixing at all
CASE_D = config([layer(2, 2, 128, 128, (32, 16), moe(36, 4, 2), v_mix=False),
                 layer(4, 1, 32, 96, (16, 8), dense(64, 1.0), v_mix=False)], width=44, vocab=50)
# E: no masks (every key stays; pages of prompts may be shared), one mixing pair
CASE_E = config([layer(4, 2, 16, 32, None, dense(64, 3.0)), layer(4, 2, 48, 32, None, moe(64, 4, 2))], width=72, vocab=75)
CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C, "D": CASE_D, "E": CASE_E}


def tensor_shapes(cfg: dict) -> dict:
    """name -> shape of every tensor of a folder of this configuration."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "pos": (cfg["max_positions"], W), "final.norm": (W,), "head": (V, W)}
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}", e["mixer"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        q = p + ".mix"
        out[p + ".norm1"] = (W,)
        out[q + ".q"], out[q + ".k"], out[q + ".v"] = (H * d, W), (G * d, W), (G * dv, W)
        out[q + ".q.norm"], out[q + ".k.norm"] = (H * d,), (G * d,)
        out[q + ".o"] = (W, H * dv)
        if m.get("v_mix"):
            out[q + ".vmix"] = ()
        mlp = e["mlp"]
        if mlp is None:
            continue
        out[p + ".norm2"] = (W,)
        if mlp["kind"] == "dense":
            out[p + ".mlp.gate"] = out[p + ".mlp.up"] = (mlp["ff"], W)
            out[p + ".mlp.down"] = (W, mlp["ff"])
        else:
            ff, E = mlp["expert"]["ff"], mlp["router"]["experts"]
            for x in range(E):
                out[f"{p}.mlp.e{x}.gate"] = out[f"{p}.mlp.e{x}.up"] = (ff, W)
                out[f"{p}.mlp.e{x}.down"] = (W, ff)
            out[p + ".mlp.router"] = (E, W)
    return out


def make_weights(cfg: dict, seed: int) -> dict:
    """bfloat16 tensors (as a folder stores them) for ``cfg``."""
    g = torch.Generator().manual_seed(seed)
    randn = lambda shape: torch.randn(shape, generator=g)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if name.endswith((".q.norm", ".k.norm")):
            t = 1.0 + 0.1 * randn(shape)
        elif last in ("norm1", "norm2", "norm"):
            t = 0.2 * randn(shape)
        elif last == "vmix":
            t = 0.2 + 0.7 * torch.rand(shape, generator=g)
        elif name == "embed":
            t = randn(shape)
        elif name == "pos":
            t = 0.5 * randn(shape)
        else:
            t = randn(shape) / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out


def safe_sequence(cfg: dict, weights: dict, n: int, seed: int):
    """(ids, float64 logits [n, vocab]) of a random sequence in which no router's choice is a close call: token by
    token, a token whose choice at some layer lies within ``CLOSE_CALL`` of turning is drawn again."""
    rng = random.Random(seed)
    w64 = {k: v.to(torch.float64) for k, v in weights.items()}
    ids, rows, state = [], [], None
    for t in range(n):
        for attempt in range(200):
            tok = rng.randrange(cfg["vocab"])
            margin = [math.inf]
            logits, new_state = plain.forward(cfg, w64, [tok], start=t, state=state, margins=margin)
            if margin[0] >= CLOSE_CALL:
                break
        else:
            raise AssertionError(f"no token without a close call at position {t}")
        ids.append(tok)
        rows.append(logits[0])
        state = new_state
    return ids, torch.stack(rows)


TOLERANCE = {"float32": 3e-5, "bfloat16": 5e-2}


def random_config(rng: random.Random) -> dict:
    """A configuration drawn at random: sizes, head counts, groupings, masks, mixing, feed-forwards, the number of layers."""
    divisor = lambda n: rng.choice([d for d in range(1, n + 1) if n % d == 0])
    width = rng.choice([40, 43, 48, 52, 64, 72, 96])
    values = rng.choice([24, 32, 48, 96])  # per token of the layers that mix theirs
    layers = []
    for _ in range(rng.randint(2, 5)):
        n = rng.randint(2, 9)
        mlp = rng.choice([None, dense(rng.choice([40, 48, 64, 90]), rng.choice([0.5, 1.0, 3.0])),
                          moe(rng.choice([24, 33, 40, 64]), n, rng.randint(1, n)), moe(rng.choice([24, 40, 64]), n, rng.randint(1, n))])
        heads = rng.choice([1, 2, 3, 4, 6, 8])
        kv = divisor(heads)
        mixing = rng.random() < 0.7 and values % kv == 0
        vdim = values // kv if mixing else rng.choice([8, 16, 20, 24, 40, 64])
        mask = None if rng.random() < 0.15 else (rng.choice([1, 5, 16, 23, 32, 64]), rng.choice([None, 1, 2, 3, 7, 12, 16, 32]))
        layers.append(layer(heads, kv, rng.choice([8, 9, 16, 24, 32, 40, 64]), vdim, mask, mlp, v_mix=mixing,
                            scale=rng.choice([None, 0.3])))
    return config(layers, width=width, vocab=rng.randint(40, 200), eps=rng.choice([1e-6, 1e-5]),
                  logit_scale=rng.choice([1.0, 0.25, 2.0]), max_positions=rng.randint(200, 300))
