"""The Lukelorn decoder as a plan.

A plain token embedding; parallel layers (one RMS norm whose weight is stored around zero, read by the mixer and the
feed-forward alike, their sum added with a factor); three kinds of mixer, chosen per layer by the configuration: grouped-query
attention (neighbouring elements rotate together, frequencies scaled by wavelength, a soft cap on the scores, a sliding window
beside which the first tokens stay visible, a sink in the softmax, an output gate per head), attention over a latent that the
heads share (queries through a latent of their own, a sliding window, an output gate per head), and a gated delta rule with a
decay per key channel (short convolutions, low-rank decay and output gate); a feed-forward that is either a gated one or a
mixture of experts without a gate (a squared ReLU; scores are sigmoids, used as they are, and multiply the experts' inputs); the
norm once more and an untied head.  A layer may run another one's tensors, with a cache or state of its own.

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.lukelorn import LukelornConfig, LukelornDense
from ..config.registry import register_architecture
from ..parts.plan import LayerPlan, ModelPlan, PartSpec, RunStep

UNIT_NORM_EPS = 1e-6  # of the delta rule's unit-length queries and keys
MAX_POSITIONS = 1 << 20  # the design sets no limit; the step function wants one


def _mixer(kind: str, m, width: int, eps: float) -> PartSpec:
    if kind == "attention":
        rotation = PartSpec("none")
        if m.rot.dims:
            scaling = None if m.rot.scaling is None else {"kind": "wavelength", **m.rot.scaling.to_dict()}
            rotation = PartSpec("scaled_rotary", {"rotary_dim": m.rot.dims, "base": m.rot.base, "layout": "interleaved",
                                                  "scaling": scaling})
        return PartSpec("gqa_attention", {
            "hidden_size": width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
            "scale": m.scale, "softcap": m.softcap, "window": m.window, "keep_first": m.keep_first, "position": rotation,
            "tensor_names": {"q": "q", "k": "k", "v": "v", "o": "o"}, "sink_name": "sink", "fp32_weights": True,
            "output_gate": {"name": "g", "kind": "sigmoid", "per_head": True}})
    if kind == "latent_attention":
        return PartSpec("latent_attention", {
            "hidden_size": width, "num_heads": m.heads, "head_dim": m.dim, "rotary_head_dim": m.rot_dim,
            "v_head_dim": m.vdim, "latent_rank": m.kv_rank, "query_rank": m.q_rank, "scale": m.scale,
            "rotary_base": m.rot.base, "rotary_dims": m.rot.dims, "rotary_layout": "interleaved", "window": m.window,
            "norm_eps": eps})
    if kind == "channel_delta":
        return PartSpec("channel_delta_rule", {
            "hidden_size": width, "num_heads": m.heads, "num_qk_heads": m.kv_heads, "head_dim": m.dim,
            "v_head_dim": m.vdim, "conv_taps": m.conv, "norm_eps": eps, "unit_norm_eps": UNIT_NORM_EPS})
    raise ValueError(kind)


def _feed_forward(mlp, width: int):
    if mlp is None:
        return None
    if isinstance(mlp, LukelornDense):
        return PartSpec("gated", {"hidden_size": width, "intermediate_size": mlp.ff, "activation": "silu"})
    return PartSpec("mixture_of_experts", {
        "hidden_size": width, "intermediate_size": mlp.ff, "experts": mlp.experts, "top": mlp.top, "router_bias_name": None,
        "sigmoid_scores": True, "input_weights": True, "gated": False, "activation": "relu2"})


def plan_lukelorn(cfg: LukelornConfig) -> ModelPlan:
    cfg.validate()
    W, unit = cfg.width, cfg.residual_mult
    # the norms of a residual stream that is held divided by ``unit``
    norm = PartSpec("grouped_rmsnorm", {"hidden_size": W, "eps": cfg.norm_eps / (unit * unit), "groups": 1, "weight_name": "",
                                        "unit_offset": True})
    layers, place = [], {}
    for i, layer in enumerate(cfg.layers):
        if cfg.owner(i) != i:
            continue
        place[i] = len(layers)
        layers.append(LayerPlan(prefix=f"l{i}", mixer=_mixer(layer.type, layer.mixer, W, cfg.norm_eps),
                                feed_forward=_feed_forward(layer.mlp, W), mixer_norm=norm, feed_forward_norm=None,
                                block=PartSpec("parallel_residual")))
    return ModelPlan(
        architecture=cfg.architecture,
        hidden_size=W,
        vocab_size=cfg.vocab,
        embedding=PartSpec("scaled_embedding", {"vocab_size": cfg.vocab, "hidden_size": W, "scale": 1.0 / unit,
                                                "weight_name": ""}),
        embedding_prefix="embed",
        layers=tuple(layers),
        run_order=tuple(RunStep(place[cfg.owner(i)]) for i in range(len(cfg.layers))),
        final_norm=norm,
        final_norm_prefix="final.norm",
        output=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": W, "tied_to": None, "weight_name": ""}),
        output_prefix="head",
        max_positions=MAX_POSITIONS,
        residual_unit=unit,
    )


register_architecture("Lukelorn", LukelornConfig, plan_lukelorn, replace=True)
