"""Attention over a latent that all heads share, as a part.

  q = y Wq^T, per head [dim plain | rot rotated];  y Wdkv^T = [c': rank | k_r: rot]
  (``query_rank``: the queries go through a latent of their own, q = (rmsnorm(y Wdq^T) * nq) Wuq^T)
  c = rmsnorm(c') * n;  k_r and each head's q_r are rotated (over the first ``rotary_dims`` of the part, elements i and
  i + rotary_dims / 2 together, or neighbours with ``rotary_layout`` "interleaved")
  per head: k = Wuk c (dim), v = Wuv c (vdim);  s = (q . k + q_r . k_r) * scale;  causal softmax;  o = sum w v
  (``window``: over the last so many keys, the token's own included)
  o_h <- o_h * sigmoid(y Wg^T)_h;  h += concat(o) Wo^T

Only [c | k_r] is cached: one row of rank + rot per token, whatever the number of heads.  The step never forms k and v
of the cached tokens.  Since q . (Wuk c) = (Wuk^T q) . c, each head's plain query is taken through Wuk^T once
(``ops.head_gemm``), the attention then runs with ONE shared key head of rank + rot whose first rank elements are
also the value (``values_in_keys``), and each head's weighted sum of latents is taken through Wuv afterwards, where
the head's output gate multiplies.  Scores, weights and sums are fp32.
"""

from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from .base import LayerCache, Mixer, PagedKV, TensorSpec
from .plan import register_part
from .position import ScaledRotary
from .recurrent import _fused_parts


class LatentAttention(Mixer):
    accepts_lazy_norm = True
    graph_safe = True
    can_overwrite = True

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, rotary_head_dim: int, v_head_dim: int,
                 latent_rank: int, scale: float, rotary_base: float, rotary_dims: int, norm_eps: float,
                 output_gate: bool = True, query_rank: Optional[int] = None, window: Optional[int] = None,
                 rotary_layout: str = "half"):
        if rotary_dims % 2 or rotary_dims > rotary_head_dim:
            raise ValueError(f"{rotary_dims} of {rotary_head_dim} dimensions cannot rotate in pairs")
        self.hidden_size, self.num_heads = int(hidden_size), int(num_heads)
        self.head_dim, self.rot, self.v_head_dim = int(head_dim), int(rotary_head_dim), int(v_head_dim)
        self.rank, self.scale = int(latent_rank), float(scale)
        self.rotary = ScaledRotary(int(rotary_dims), float(rotary_base), rotary_layout)
        self.query_rank = None if query_rank is None else int(query_rank)
        self.window = None if window is None else int(window)
        if (self.query_rank is not None and self.query_rank <= 0) or (self.window is not None and self.window <= 0):
            raise ValueError(f"a query latent of {query_rank}, a window of {window}: positive counts are needed")
        self.norm_eps, self.output_gate = float(norm_eps), bool(output_gate)
        self.q_size = self.num_heads * (self.head_dim + self.rot)
        self.row = self.rank + self.rot  # a token's cache row, and the size of a head's query in the attention
        if self.row > 1024:
            raise ValueError(f"cache rows of {self.row} are larger than the attention kernel takes (1024)")

    def tensor_specs(self, prefix):
        H, nh = self.hidden_size, self.num_heads
        if self.query_rank is None:
            specs = [TensorSpec(f"{prefix}.q", (self.q_size, H), "matrix")]
        else:
            specs = [TensorSpec(f"{prefix}.dq", (self.query_rank, H), "matrix"),
                     TensorSpec(f"{prefix}.dq.norm", (self.query_rank,), "norm"),
                     TensorSpec(f"{prefix}.uq", (self.q_size, self.query_rank), "matrix")]
        specs += [
            TensorSpec(f"{prefix}.dkv", (self.row, H), "matrix"),
            TensorSpec(f"{prefix}.dkv.norm", (self.rank,), "norm"),
            TensorSpec(f"{prefix}.uk", (nh * self.head_dim, self.rank), "matrix"),
            TensorSpec(f"{prefix}.uv", (nh * self.v_head_dim, self.rank), "matrix"),
        ]
        if self.output_gate:
            specs.append(TensorSpec(f"{prefix}.g", (nh, H), "matrix"))
        return specs + [TensorSpec(f"{prefix}.o", (H, nh * self.v_head_dim), "matrix")]

    def bind(self, tensors, prefix):
        nh = self.num_heads
        first = tensors.pop(f"{prefix}.q" if self.query_rank is None else f"{prefix}.dq")
        parts = [first, tensors.pop(f"{prefix}.dkv")]
        if self.output_gate:
            parts.append(tensors.pop(f"{prefix}.g"))
        self.in_weight, offsets = _fused_parts(parts)  # [q or its latent | dkv | gate], each from a multiple of eight rows on
        self.dkv_off, self.gate_off = offsets[1], offsets[-1]
        if self.query_rank is not None:
            self.q_norm = tensors[f"{prefix}.dq.norm"]
            self.uq = tensors[f"{prefix}.uq"]
            pad = (-self.query_rank) % 8  # zero columns meet zeros: the product's rows then start on 16 bytes
            self.q_cols = self.query_rank + pad
            if pad:
                self.uq = torch.cat([self.uq, self.uq.new_zeros(self.q_size, pad)], dim=1).contiguous()
        self.latent_norm = tensors[f"{prefix}.dkv.norm"]
        # per head [K, N]: the key up-projection as stored ([dim, rank]); the value one transposed ([rank, vdim])
        self.uk = tensors.pop(f"{prefix}.uk").reshape(nh, self.head_dim, self.rank).contiguous()
        self.uv = tensors.pop(f"{prefix}.uv").reshape(nh, self.v_head_dim, self.rank).transpose(1, 2).contiguous()
        self.o_weight = tensors[f"{prefix}.o"]

    def cache_need(self):
        # one shared key head; the value is the key's first ``rank`` elements, so no value rows are kept
        return PagedKV(1, self.row, self.window, 0)

    def forward(self, x, h, ctx, cache: LayerCache, owns_cache: bool, accumulate: bool = True):
        T = x.shape[0]
        nh, d, r, dv, rank, row = self.num_heads, self.head_dim, self.rot, self.v_head_dim, self.rank, self.row
        ws = ctx.workspace
        meta = ctx.paged[cache.group]
        proj = ws.get("latent_in", (T, self.in_weight.shape[0]), ctx.act_dtype)
        ops.gemm(x, self.in_weight, None, proj)
        q_att = ws.get("latent_queries", (T, nh * row), ctx.act_dtype)
        table = self.rotary.table(proj.device)
        keys = None
        if owns_cache:
            keys = (proj[:, self.dkv_off:self.dkv_off + row], self.latent_norm, meta.slot_mapping, cache.k)
        if self.query_rank is None:
            q = proj[:, :self.q_size]
            ops.latent_prepare(ctx.positions, table, self.norm_eps, nh, d, r, rank, queries=(q, q_att), keys=keys)
        else:
            latent = proj[:, :self.query_rank]  # normed in place (the columns that fill it up stay zero)
            ops.latent_prepare(ctx.positions, table, self.norm_eps, nh, d, r, rank, keys=keys,
                               q_latent=(latent, self.q_norm, latent))
            q = ws.get("latent_q", (T, self.q_size), ctx.act_dtype)
            ops.gemm(proj[:, :self.q_cols], self.uq, None, q)
            ops.latent_prepare(ctx.positions, table, self.norm_eps, nh, d, r, rank, queries=(q, q_att))
        ops.head_gemm(q, d + r, self.uk, q_att, row)  # the plain queries through the key up-projection
        mixed = ws.get("latent_mixed", (T, nh * rank), ctx.act_dtype)
        ops.paged_attention(q_att, mixed, cache.k, None, meta.block_tables, ctx, nh, 1, row, self.window or 0, self.scale,
                            v_head_dim=rank, values_in_keys=True)
        out = ws.get("latent_out", (T, nh * dv), ctx.act_dtype)
        gate = proj[:, self.gate_off:self.gate_off + nh] if self.output_gate else None
        ops.head_gemm(mixed, rank, self.uv, out, dv, gate=gate)
        ops.gemm(out, self.o_weight, None, h, accumulate=accumulate)


register_part("mixer", "latent_attention", LatentAttention)
