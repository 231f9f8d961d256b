"""The Retezen decoder as a plan.

A token embedding plus a learned vector per position; layers whose norms stand on the sublayers' outputs (the sublayers
read the residual stream itself, the norm's weight is stored around zero and multiplies as 1 + w); grouped-query
attention without rotation, whose queries and keys are RMS-normed over their whole projection, in which a token sees a
sliding window of tokens and, beside it, one pooled key and value (means) for every block of positions that lies wholly
before the window, and whose values are mixed with those of the first layer that says so; a feed-forward that is either a
gated one with a clamped gate or a mixture of experts (scores are sigmoids, used as they are, and multiply the experts'
inputs); the norm once more and an untied head with a factor on the logits.

Tensor names: ``embed``, ``pos``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.retezen import RetezenConfig, RetezenDense
from ..parts.plan import LayerPlan, ModelPlan, PartSpec, RunStep


def _feed_forward(mlp, width: int):
    if mlp is None:
        return None
    if isinstance(mlp, RetezenDense):
        return PartSpec("gated", {"hidden_size": width, "intermediate_size": mlp.ff, "activation": "clamped_swish",
                                  "limit": mlp.limit})
    return PartSpec("mixture_of_experts", {
        "hidden_size": width, "intermediate_size": mlp.ff, "experts": mlp.experts, "top": mlp.top,
        "router_bias_name": None, "sigmoid_scores": True, "input_weights": True, "activation": "silu"})


def plan_retezen(cfg: RetezenConfig) -> ModelPlan:
    cfg.validate()
    W = cfg.width
    norm = PartSpec("grouped_rmsnorm", {"hidden_size": W, "eps": cfg.norm_eps, "groups": 1, "weight_name": "",
                                        "unit_offset": True})
    mixing = [i for i, layer in enumerate(cfg.layers) if layer.mixer.v_mix]
    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        mixer = PartSpec("gqa_attention", {
            "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
            "scale": m.scale, "window": m.window, "pool": m.pool, "position": PartSpec("none"),
            "qk_norm": {"eps": cfg.norm_eps, "q": "q.norm", "k": "k.norm"}, "fp32_weights": True,
            "tensor_names": {"q": "q", "k": "k", "v": "v", "o": "o"},
            "value_mix": {"lambda": "vmix", "role": "source" if i == mixing[0] else "mix"} if m.v_mix else None})
        layers.append(LayerPlan(prefix=f"l{i}", mixer=mixer, feed_forward=_feed_forward(layer.mlp, W), mixer_norm=norm,
                                feed_forward_norm=norm, block=PartSpec("output_norm")))
    return ModelPlan(
        architecture=cfg.architecture,
        hidden_size=W,
        vocab_size=cfg.vocab,
        embedding=PartSpec("learned_position_embedding", {"vocab_size": cfg.vocab, "hidden_size": W,
                                                          "max_positions": cfg.max_positions, "weight_name": "",
                                                          "position_name": "pos"}),
        embedding_prefix="embed",
        layers=tuple(layers),
        run_order=tuple(RunStep(i) for i in range(len(layers))),
        final_norm=norm,
        final_norm_prefix="final.norm",
        output=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": W, "tied_to": None, "weight_name": "",
                                        "logit_scale": cfg.logit_scale}),
        output_prefix="head",
        max_positions=cfg.max_positions,
        positions_bounded=True,
        extra={"ignorable_tensors": tuple(f"l{i}.mix.vmix" for i, layer in enumerate(cfg.layers) if not layer.mixer.v_mix)},
    )


register_architecture("Retezen", RetezenConfig, plan_retezen, replace=True)
