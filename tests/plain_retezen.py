"""A plain, slow restatement of the Retezen decoder, one function per mechanism, in one precision throughout
(float64 by default).  It shares no code with the package: it takes the dict of config.json and a dict of
tensors by name, loops over tokens where that is the clearest way to say what is computed, and continues a
sequence from an explicit state, so that the plain implementation itself can be checked cut anywhere.

Notation: W is the model width, t a position counted from 0 in its sequence, S the window, P the block size.

  embedding        x_t = E[id_t] + pos[t]
  norm             n(x, w) = x / sqrt(mean(x^2) + eps) * (1 + w)
  layer            x <- x + n(mixer(x), w1);  x <- x + n(ff(x), w2)    (the sublayers read x itself)
  attention        q, k, v = Wq x, Wk x, Wv x; q <- q / sqrt(mean(q^2) + eps) * nq over the WHOLE projection (all heads
                   at once), k likewise; head h reads kv head floor(h / (heads / kv heads)); no rotation
  value mixing     in a layer with v_mix other than the first one: v <- (1 - lam) v + lam v1, v1 the first such layer's
                   values of the same token (before any mixing there is none)
  visible          the tokens j with 0 <= t - j < S, and beside them one key and value for every block b of P tokens
                   (positions bP .. bP + P - 1) with bP + P - 1 <= t - S: the means of the block's P keys and P values;
                   one softmax over both, scores (q . k) * scale
  dense            g = min(Wg x, L), u = clamp(Wu x, -L, L);  Wd (g sigmoid(1.702 g) (u + 1))
  mixture          s = sigmoid(Wr x); the `top` largest s;  sum over the chosen e of expert_e(s_e x),
                   expert(z) = Wd (silu(Wg z) * (Wu z))
  output           logits = (head n(x, final)) * logit_scale
"""

from __future__ import annotations

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def embedding(w, ids, start=0):
    ids = torch.as_tensor(list(ids), dtype=torch.long)
    return w["embed"][ids] + w["pos"][start:start + len(ids)]


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def visible(t, mask):
    """(positions of the tokens that the query at ``t`` sees, blocks that it sees); mask None: every token up to t."""
    if not mask:
        return list(range(t + 1)), []
    size, pool = mask["size"], mask.get("pool")
    tokens = [j for j in range(t + 1) if t - j < size]
    blocks = []
    if pool:
        b = 0
        while b * pool + pool - 1 <= t - size:
            blocks.append(b)
            b += 1
    return tokens, blocks


def keys_and_values_seen(k, v, t, mask):
    """k, v [t + 1 or more, ...]: the rows that the query at ``t`` meets, pooled blocks first."""
    tokens, blocks = visible(t, mask)
    rows_k = [k[b * mask["pool"]:(b + 1) * mask["pool"]].mean(dim=0) for b in blocks] + [k[j] for j in tokens]
    rows_v = [v[b * mask["pool"]:(b + 1) * mask["pool"]].mean(dim=0) for b in blocks] + [v[j] for j in tokens]
    return torch.stack(rows_k), torch.stack(rows_v)


def attend(q, k, v, positions, mixer):
    """q [T, H, d] of the tokens at ``positions``; k, v [positions seen so far, G, .] as cached.  Returns [T, H, dv]."""
    H, G = mixer["heads"], mixer["kv_heads"]
    out = torch.zeros(q.shape[0], H, v.shape[-1], dtype=q.dtype)
    for n, t in enumerate(positions):
        ks, vs = keys_and_values_seen(k, v, t, mixer.get("mask"))
        for h in range(H):
            g = h // (H // G)
            p = torch.softmax((ks[:, g] @ q[n, h]) * mixer["scale"], dim=0)
            out[n, h] = p @ vs[:, g]
    return out


def attention(x, w, prefix, mixer, eps, start=0, past=None, first_values=None):
    """``past`` = (keys, values) of the positions before ``start`` as cached, or None.  ``first_values``: the first mixing
    layer's values of these tokens [T, G dv], or None where nothing is mixed.  Returns (out, (keys, values), the
    layer's own values before any mixing)."""
    H, G, d, dv = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    T = x.shape[0]
    q = rms(x @ w[prefix + ".q"].T, eps) * w[prefix + ".q.norm"]
    k = rms(x @ w[prefix + ".k"].T, eps) * w[prefix + ".k.norm"]
    own = x @ w[prefix + ".v"].T
    v = own if first_values is None else mix_values(own, first_values, w[prefix + ".vmix"])
    q, k, v = q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, dv)
    if past is not None:
        k, v = torch.cat([past[0], k]), torch.cat([past[1], v])
    o = attend(q, k, v, range(start, start + T), mixer)
    return o.reshape(T, H * dv) @ w[prefix + ".o"].T, (k, v), own


def dense(x, w, prefix, limit):
    g = torch.clamp(x @ w[prefix + ".gate"].T, max=limit)
    u = torch.clamp(x @ w[prefix + ".up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[prefix + ".down"].T


def router(x, w, prefix, mlp, margins=None):
    """(chosen experts, their scores) of every row.  ``margins`` (a list with one entry per token, or None): lowered to
    the gap between the last chosen logit and the first that is not, over the size a logit has (the row's root mean square
    times that of the router rows' lengths; the logits' own spread says nothing where there are two), where that is smaller."""
    E, top = mlp["router"]["experts"], mlp["router"]["top"]
    z = x @ w[prefix + ".router"].T
    if margins is not None and top < E:
        ordered = torch.sort(z, dim=-1, descending=True).values
        size = (x * x).mean(dim=-1).sqrt() * (w[prefix + ".router"] ** 2).sum(dim=-1).mean().sqrt()
        gap = (ordered[:, top - 1] - ordered[:, top]) / size
        for t in range(x.shape[0]):
            margins[t] = min(margins[t], float(gap[t]))
    s = torch.sigmoid(z)
    chosen = [sorted(range(E), key=lambda e: -float(z[t, e]))[:top] for t in range(x.shape[0])]
    return chosen, [[s[t, e] for e in chosen[t]] for t in range(x.shape[0])]


def expert(z, w, prefix):
    return w[prefix + ".down"] @ (silu(w[prefix + ".gate"] @ z) * (w[prefix + ".up"] @ z))


def mixture(x, w, prefix, mlp, margins=None):
    chosen, weights = router(x, w, prefix, mlp, margins)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e, s in zip(chosen[t], weights[t]):
            out[t] += expert(s * x[t], w, f"{prefix}.e{e}")
    return out


def feed_forward(x, w, prefix, mlp, margins=None):
    if mlp["kind"] == "dense":
        return dense(x, w, prefix, mlp["limit"])
    if mlp["kind"] == "moe":
        return mixture(x, w, prefix, mlp, margins)
    raise ValueError(mlp["kind"])


def forward(cfg, w, ids, start=0, state=None, dtype=torch.float64, after_layer=None, margins=None):
    """Logits [len(ids), vocab] of the tokens ``ids`` at positions start .. and the state to continue from.
    ``state``: what an earlier call returned (keys and values of every layer), or None at position 0.
    ``after_layer(i, x)`` sees the residual stream after every layer; ``margins``: see ``router``."""
    w = {k: t.to(dtype) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = embedding(w, ids, start)
    new_state, first_values = [], None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        if layer["type"] != "attention":
            raise ValueError(layer["type"])
        mixing = bool(layer["mixer"].get("v_mix"))
        m, s, own = attention(x, w, p + ".mix", layer["mixer"], eps, start, None if state is None else state[i],
                              first_values if mixing else None)
        if mixing and first_values is None:
            first_values = own
        new_state.append(s)
        x = x + norm(m, w[p + ".norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + norm(feed_forward(x, w, p + ".mlp", layer["mlp"], margins), w[p + ".norm2"], eps)
        if after_layer is not None:
            after_layer(i, x)
    return norm(x, w["final.norm"], eps) @ w["head"].T * cfg.get("logit_scale", 1.0), new_state
