"""The Lukelorn decoder once more, plainly: one function per mechanism, float64 torch on the CPU, a whole sequence at a
time (or portion by portion through explicit states), sharing no code with the package.

Notation: a sequence of T tokens is a [T, ...] tensor; weights are a dict name -> tensor as the folder names them;
``cfg`` is the dict of config.json.  Every function takes what it needs explicitly.
"""

from __future__ import annotations

import math

import torch

F = torch.float64
UNIT_EPS = 1e-6


def rms_div(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    return rms_div(x, eps) * (1.0 + w)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + torch.clamp(x, min=0.0)


# --------------------------------------------------------------------------------------------- positions
def frequencies(dims, base, scaling=None):
    """base^(-2 i / dims); with ``scaling`` (factor, low, high, original) waves longer than original / low are slowed down
    by the factor, those shorter than original / high stay, those between get a mixture."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            wave = 2.0 * math.pi / f
            low, high, original = scaling["low"], scaling["high"], scaling["original"]
            if wave > original / low:
                f = f / scaling["factor"]
            elif not wave < original / high:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F)


def rotate_pairs(x, positions, freq):
    """x [T, n, d]: the elements 2i and 2i + 1 of each vector turned by position * freq[i]; the rest passes."""
    a = torch.as_tensor(positions, dtype=F)[:, None] * freq[None]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    n = 2 * freq.numel()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


# --------------------------------------------------------------------------------------------- softmax attention
def seen(T, S, size=None, keep_first=0):
    """[T, S] bool: which of S keys the last T of their positions see.  ``size``: the newest ``size`` keys (None: all), and
    beside them the first ``keep_first`` of the sequence."""
    i = torch.arange(T)[:, None] + (S - T)
    j = torch.arange(S)[None, :]
    ok = j <= i
    if size is not None:
        ok = ok & ((i - j < size) | (j < keep_first))
    return ok


def weighted_values(scores, visible, v, sink=None):
    """softmax(scores [H, T, S]) v [S, H, dv]; ``sink`` [H]: one more exponential in the denominator."""
    H, T, S = scores.shape
    scores = scores.masked_fill(~visible[None], float("-inf"))
    if sink is not None:
        scores = torch.cat([scores, sink[:, None, None].expand(H, T, 1)], dim=-1)
    return torch.einsum("hts,shv->thv", torch.softmax(scores, dim=-1)[..., :S], v)


def capped(scores, cap):
    return scores if cap is None else cap * torch.tanh(scores / cap)


def attention(h, w, p, m, positions, past=None):
    """``past``: (keys [P, G, d], values [P, G, dv]) of every token before h[0]."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    freq = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    q = rotate_pairs((h @ w[p + ".q"].T).reshape(T, H, d), positions, freq)
    k = rotate_pairs((h @ w[p + ".k"].T).reshape(T, G, d), positions, freq)
    v = (h @ w[p + ".v"].T).reshape(T, G, dv)
    if past is not None:
        k, v = torch.cat([past[0], k]), torch.cat([past[1], v])
    kv_of = torch.arange(H) // (H // G)
    scores = capped(torch.einsum("thd,shd->hts", q, k[:, kv_of]) * m["scale"], m.get("softcap"))
    mask = m.get("mask") or {}
    visible = seen(T, k.shape[0], mask.get("size"), mask.get("keep_first", 0))
    o = weighted_values(scores, visible, v[:, kv_of], w[p + ".sink"])
    o = o * torch.sigmoid(h @ w[p + ".g"].T)[..., None]
    return o.reshape(T, H * dv) @ w[p + ".o"].T, (k, v)


def latent_attention(h, w, p, m, eps, positions, past=None):
    """``past``: (latents [P, rank], rotated key parts [P, rot]) of every token before h[0]."""
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_div(h @ w[p + ".dq"].T, eps) * w[p + ".dq.norm"]
    q = (cq @ w[p + ".uq"].T).reshape(T, H, d + r)
    dkv = h @ w[p + ".dkv"].T
    c = rms_div(dkv[:, :rank], eps) * w[p + ".dkv.norm"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    freq = frequencies(rot["dims"], rot["base"])
    q_rot = rotate_pairs(q[..., d:], positions, freq)
    k_rot = rotate_pairs(dkv[:, None, rank:], positions, freq)[:, 0]
    if past is not None:
        c, k_rot = torch.cat([past[0], c]), torch.cat([past[1], k_rot])
    S = c.shape[0]
    k = (c @ w[p + ".uk"].T).reshape(S, H, d)
    v = (c @ w[p + ".uv"].T).reshape(S, H, dv)
    scores = (torch.einsum("thd,shd->hts", q[..., :d], k) + torch.einsum("thr,sr->hts", q_rot, k_rot)) * m["scale"]
    o = weighted_values(scores, seen(T, S, (m.get("mask") or {}).get("size")), v)
    o = o * torch.sigmoid(h @ w[p + ".g"].T)[..., None]
    return o.reshape(T, H * dv) @ w[p + ".o"].T, (c, k_rot)


# --------------------------------------------------------------------------------------------- recurrence
def causal_conv(x, w, before=None):
    """Per channel: out_t = sum_j w[:, j] x_(t - taps + 1 + j).  ``before`` [taps - 1, C]: the inputs ahead of x[0]."""
    T, C = x.shape
    taps = w.shape[1]
    full = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype) if before is None else before, x])
    out = torch.zeros_like(x)
    for j in range(taps):
        out = out + full[j:j + T] * w[:, j]
    return out, full[full.shape[0] - (taps - 1):].clone()


def channel_delta_scan(q, k, v, g, beta, S):
    """Per head: S <- diag(g_t) S; u = beta_t (v_t - S^T k_t); S <- S + k_t u^T; o_t = S^T q_t.
    q, k [T, H, n]; v [T, H, dv]; g [T, H, n]; beta [T, H]; S [H, n, dv]."""
    S = S.clone()
    o = torch.zeros(v.shape, dtype=F)
    for t in range(q.shape[0]):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hnv,hn->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hnv,hn->hv", S, q[t])
    return o, S


def channel_decay(h, w, p, heads, dim):
    z = (h @ w[p + ".a1"].T) @ w[p + ".a2"].T + w[p + ".dt_bias"]
    return torch.exp(-torch.exp(w[p + ".A_log"])[:, None] * softplus(z).reshape(-1, heads, dim))


def channel_delta(h, w, p, m, eps, past=None):
    """``past``: (state [heads, dim, vdim], the three convolutions' last inputs) or None."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rows, befores = {}, []
    for i, n in enumerate("qkv"):
        y, b = causal_conv(h @ w[f"{p}.{n}"].T, w[f"{p}.{n}.conv"], None if past is None else past[1][i])
        rows[n] = silu(y)
        befores.append(b)
    unit = lambda x: x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + UNIT_EPS)
    head_of = torch.arange(H) // (H // G)
    q = unit(rows["q"].reshape(T, G, d))[:, head_of] * d ** -0.5
    k = unit(rows["k"].reshape(T, G, d))[:, head_of]
    v = rows["v"].reshape(T, H, dv)
    beta = torch.sigmoid(h @ w[p + ".b"].T)
    S = torch.zeros(H, d, dv, dtype=F) if past is None else past[0]
    o, S = channel_delta_scan(q, k, v, channel_decay(h, w, p, H, d), beta, S)
    gate = torch.sigmoid((h @ w[p + ".g1"].T) @ w[p + ".g2"].T).reshape(T, H, dv)
    o = rms_div(o, eps) * w[p + ".norm"] * gate
    return o.reshape(T, H * dv) @ w[p + ".o"].T, (S, befores)


# --------------------------------------------------------------------------------------------- feed-forward
def dense(h, w, p):
    return (silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def router(h, w, p, top):
    """(chosen experts [T, top], their scores [T, top], how far the closest choice was from turning, per token)."""
    z = h @ w[p + ".router"].T
    s = torch.sigmoid(z)
    best, idx = torch.sort(z, dim=-1, descending=True, stable=True)
    margin = best[:, top - 1] - best[:, top] if top < z.shape[1] else torch.full((z.shape[0],), math.inf, dtype=F)
    chosen = idx[:, :top]
    return chosen, torch.gather(s, 1, chosen), margin


def expert(x, w, p):
    return torch.clamp(x @ w[p + ".up"].T, min=0.0) ** 2 @ w[p + ".down"].T


def mixture(h, w, p, mlp, margins=None):
    chosen, weights, margin = router(h, w, p, mlp["router"]["top"])
    if margins is not None:
        margins[0] = min(margins[0], float(margin.min()))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), weights[t]):
            out[t] += expert(s * h[t:t + 1], w, f"{p}.e{e}")[0]
    return out


# --------------------------------------------------------------------------------------------- the decoder
def forward(cfg, w, tokens, start=0, state=None, margins=None, after=None):
    """Logits [T, vocab] of the tokens at positions ``start``.. and the state after them (None at a sequence's start).
    ``margins`` [x]: gets the smallest distance of a router's choice from turning; ``after``: a list that gets the
    residual stream after every layer."""
    eps, mult = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    positions = torch.arange(start, start + len(tokens))
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    state = state or [None] * len(cfg["layers"])
    new = []
    for i, e in enumerate(cfg["layers"]):
        j = i
        while cfg["layers"][j].get("weights_of") is not None:
            j = cfg["layers"][j]["weights_of"]
        p, m = f"l{j}", e["mixer"]
        h = norm_around_zero(x, w[p + ".norm1"], eps)
        if e["type"] == "attention":
            y, s = attention(h, w, p + ".mix", m, positions, state[i])
        elif e["type"] == "latent_attention":
            y, s = latent_attention(h, w, p + ".mix", m, eps, positions, state[i])
        else:
            y, s = channel_delta(h, w, p + ".mix", m, eps, state[i])
        new.append(s)
        if e.get("mlp") is not None:
            y = y + (dense(h, w, p + ".mlp") if e["mlp"]["kind"] == "dense" else mixture(h, w, p + ".mlp", e["mlp"], margins))
        x = x + mult * y
        if after is not None:
            after.append(x)
    return norm_around_zero(x, w["final.norm"], eps) @ w["head"].T, new
