"""Small Lukelorn configurations and weights for the tests (see ``netinex_cases`` for how rows are compared).

Projections are drawn with a standard deviation of 1 / sqrt(inputs), scores so large that the soft caps bend them, sinks and
gates of order one, decays from a few tokens to hundreds, router matrices so that the experts' logits spread over a few units,
so that every mechanism moves the logits by far more than a tolerance.  Sequences are drawn token by token so that no router's
choice is a close call anywhere (``safe_sequence``)."""

from __future__ import annotations

import math
import random

import torch

import plain_lukelorn as plain
from netinex_cases import random_ids, row_errors  # noqa: F401 (shared with the tests)

CLOSE_CALL = 0.12  # of a router's logits, which spread over a few units


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


SCALING = {"factor": 3.0, "low": 1.0, "high": 5.0, "original": 96.0}


def attention(heads, kv_heads, dim, vdim, mask, mlp, rot=None, base=700.0, scaling=SCALING, softcap=4.0, scale=None):
    """``mask``: (window, kept first tokens) or None."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
         "scale": scale if scale is not None else 2.5 / math.sqrt(dim)}
    r = dim - dim % 2 if rot is None else rot
    if r:
        m["rot"] = {"base": base, "dims": r}
        if scaling is not None:
            m["rot"]["scaling"] = dict(scaling)
    if softcap is not None:
        m["softcap"] = softcap
    if mask is not None:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, mlp, base=300.0, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "scale": scale if scale is not None else 2.0 / math.sqrt(dim + rot_dim)}
    if rot_dim:
        m["rot"] = {"base": base, "dims": rot_dim}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": mlp}


def again(layers, i):
    """One more run of layer i's tensors."""
    return dict(layers[i], weights_of=i)


def config(layers, width=64, vocab=97, eps=1e-6, mult=0.4):
    return {"architecture": "Lukelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": layers}


def _case_a():
    first = [latent(4, 16, 8, 24, 40, 48, 19, dense(96)), attention(4, 2, 32, 32, (24, 5), moe(40, 6, 1)),
             delta(4, 2, 16, 24, 4, moe(40, 6, 1))]
    return config(first + [again(first, 1), again(first, 0), again(first, 2)], mult=0.8)


def _case_b():
    """Values of other sizes than keys, part of a head rotated, frequencies as they are, more kept tokens than a page and than
    the window, inner sizes that are no multiple of eight, several experts, a factor of one, a layer without a feed-forward,
    tensors that run three times by way of one another."""
    first = [attention(6, 3, 24, 20, (11, 35), moe(56, 7, 3), rot=16, scaling=None, softcap=2.0), delta(3, 1, 40, 20, 3, dense(72)),
             latent(3, 24, 6, 16, 27, 33, 30, moe(33, 5, 2)), attention(4, 1, 16, 16, (40, 3), None, base=50.0)]
    layers = first + [again(first, 2), again(first, 3)]
    layers.append(dict(again(first, 2), weights_of=4))
    layers.append(again(first, 1))
    return config(layers, width=48, vocab=131, eps=1e-5, mult=1.0)


def _case_c():
    """Sizes that are no multiple of two, windows of one token, one kept token, one tap, all experts chosen, no rotation."""
    return config([attention(3, 3, 15, 9, (1, 1), moe(33, 3, 3), rot=4), latent(3, 9, 2, 7, 5, 13, 1, dense(50)),
                   delta(3, 3, 15, 9, 1, moe(24, 9, 4)), delta(2, 1, 33, 5, 2, None), attention(2, 1, 33, 27, (7, 0), dense(31), rot=0),
                   latent(5, 11, 0, 10, 12, 21, 4, None)], width=43, vocab=61, eps=1e-5, mult=1.7)


def _case_d():
    """Heads of 64 and 128, windows and kept tokens at page borders exactly, a width that is no multiple of eight."""
    first = [attention(2, 2, 128, 128, (32, 16), moe(36, 4, 1)), latent(2, 32, 16, 64, 64, 112, 16, dense(64)),
             delta(2, 2, 64, 64, 4, moe(64, 4, 2)), attention(8, 2, 64, 64, (16, 32), dense(48), softcap=10.0)]
    return config(first + [again(first, 0)], width=44, vocab=50, mult=0.25)


def _case_e():
    """No masks and no caps."""
    return config([attention(4, 2, 16, 32, None, dense(64), softcap=None), latent(4, 16, 16, 16, 24, 32, None, moe(64, 4, 2))],
                  width=72, vocab=75, mult=0.6)


CASES = {"A": _case_a(), "B": _case_b(), "C": _case_c(), "D": _case_d(), "E": _case_e()}
LOW_RANKS = {"A": (24, 8), "B": (5, 16), "C": (3, 1), "D": (16, 40), "E": (8, 8)}  # inner sizes of decay and output gate


def mixer_shapes(kind: str, m: dict, W: int, ranks: tuple) -> dict:
    H = m["heads"]
    if kind == "attention":
        G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
        return {"q": (H * d, W), "k": (G * d, W), "v": (G * dv, W), "sink": (H,), "g": (H, W), "o": (W, H * dv)}
    if kind == "latent_attention":
        d, r, dv, qr, kr = m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
        return {"dq": (qr, W), "dq.norm": (qr,), "uq": (H * (d + r), qr), "dkv": (kr + r, W), "dkv.norm": (kr,),
                "uk": (H * d, kr), "uv": (H * dv, kr), "g": (H, W), "o": (W, H * dv)}
    G, d, dv, taps = m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    out = {}
    for n, size in (("q", G * d), ("k", G * d), ("v", H * dv)):
        out[n], out[n + ".conv"] = (size, W), (size, taps)
    out.update({"b": (H, W), "A_log": (H,), "norm": (dv,), "a1": (ranks[0], W), "a2": (H * d, ranks[0]), "dt_bias": (H * d,),
                "g1": (ranks[1], W), "g2": (H * dv, ranks[1]), "o": (W, H * dv)})
    return out


def tensor_shapes(cfg: dict, ranks=(16, 16)) -> dict:
    """name -> shape of every tensor of a folder of this configuration."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, e in enumerate(cfg["layers"]):
        if e.get("weights_of") is not None:
            continue
        p = f"l{i}"
        out[p + ".norm1"] = (W,)
        out.update({f"{p}.mix.{n}": s for n, s in mixer_shapes(e["type"], e["mixer"], W, ranks).items()})
        mlp = e["mlp"]
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            out[p + ".mlp.gate"] = out[p + ".mlp.up"] = (mlp["ff"], W)
            out[p + ".mlp.down"] = (W, mlp["ff"])
        else:
            ff, E = mlp["expert"]["ff"], mlp["router"]["experts"]
            for x in range(E):
                out[f"{p}.mlp.e{x}.up"], out[f"{p}.mlp.e{x}.down"] = (ff, W), (W, ff)
            out[p + ".mlp.router"] = (E, W)
    return out


def draw(name: str, shape, g) -> torch.Tensor:
    randn = lambda: torch.randn(shape, generator=g)
    last = name.rsplit(".", 1)[-1]
    if last == "norm1" or name == "final.norm":
        return 0.2 * randn()
    if last == "norm":
        return 1.0 + 0.1 * randn()
    if last == "A_log":
        return 0.5 * randn()
    if last == "dt_bias":
        return -5.0 + 6.0 * torch.rand(shape, generator=g)
    if last == "sink":
        return 1.0 + randn()
    if last == "conv":
        return randn() / math.sqrt(shape[-1])
    if last == "router":
        return 2.0 * randn() / math.sqrt(shape[-1])
    if name == "embed":
        return randn()
    return randn() / math.sqrt(shape[-1])


def make_weights(cfg: dict, seed: int, ranks=(16, 16)) -> dict:
    """bfloat16 tensors (as a folder stores them) for ``cfg``."""
    g = torch.Generator().manual_seed(seed)
    return {name: draw(name, shape, g).to(torch.bfloat16) for name, shape in tensor_shapes(cfg, ranks).items()}


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
    """A configuration drawn at random: mixers, sizes, head counts, groupings, masks, feed-forwards, layers run again."""
    divisor = lambda n: rng.choice([d for d in range(1, n + 1) if n % d == 0])
    layers = []
    for _ in range(rng.randint(2, 5)):
        n = rng.randint(2, 9)
        mlp = rng.choice([None, dense(rng.choice([40, 48, 64, 90])), moe(rng.choice([24, 33, 40, 64]), n, 1),
                          moe(rng.choice([24, 40, 64]), n, rng.randint(1, n))])
        heads = rng.choice([1, 2, 3, 4, 6, 8])
        kind = rng.choice(["attention", "latent", "delta"])
        if kind == "attention":
            dim = rng.choice([8, 9, 16, 24, 32, 40, 64])
            mask = None if rng.random() < 0.15 else (rng.choice([1, 5, 16, 23, 32, 64]), rng.choice([0, 1, 3, 16, 17, 40]))
            layers.append(attention(heads, divisor(heads), dim, rng.choice([dim, 8, 20, 24, 40]), mask, mlp,
                                    rot=rng.choice([None, 0, 4, 8]), base=rng.choice([50.0, 1e4]),
                                    scaling=rng.choice([None, SCALING, {"factor": 8.0, "low": 0.5, "high": 2.0, "original": 40.0}]),
                                    softcap=rng.choice([None, 1.5, 6.0, 40.0]), scale=rng.choice([None, 0.3])))
        elif kind == "latent":
            layers.append(latent(heads, rng.choice([8, 13, 16, 32]), rng.choice([0, 2, 8, 16]), rng.choice([8, 9, 24, 32]),
                                 rng.choice([12, 24, 37, 64]), rng.choice([16, 21, 48, 96]), rng.choice([None, 1, 9, 16, 33]), mlp))
        else:
            layers.append(delta(heads, divisor(heads), rng.choice([8, 12, 16, 33]), rng.choice([8, 9, 20, 32]), rng.randint(1, 5), mlp))
        if len(layers) > 1 and rng.random() < 0.4:
            i = rng.randrange(len(layers))
            layers.append(dict(layers[i], weights_of=i))
    return config(layers, width=rng.choice([40, 43, 48, 52, 64, 72, 96]), vocab=rng.randint(40, 200),
                  eps=rng.choice([1e-6, 1e-5]), mult=rng.choice([0.2, 0.5, 1.0, 1.5]))
