"""Zabusun as a :class:`ModelSpec`.

The embedding rows are normed as they enter the residual sum.  Every layer is an ``output_norm`` block: the sublayers read the sum as it
is, and what an RMS norm makes of their outputs is added.  The mixer is ``weighted_mixers`` of a ``gqa_attention`` (q and k normed per
head, then partly rotated in halves with YaRN-scaled frequencies; sigmoid weights with a learnt number per head added to the scores; a
gate per head) beside a ``min_gru``; the feed-forward is a ``clamped_glu``, an ``expert_mixture`` of such units (sigmoid scores, not
renormalised, that weigh an expert's input) or none.  The head is the embedding table.  Tensor names: ``embed``, ``embed.norm``,
``l<i>.norm1`` / ``norm2``, ``l<i>.mix.left.*`` / ``right.*``, ``l<i>.mlp.*``, ``final.norm``.
"""
from __future__ import annotations

from typing import Optional

from pylon_b200.config.model_config import ZabusunConfig, ZabusunLayer
from pylon_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, RunSpec

MAX_POSITIONS = 1 << 20    # no learnt table limits a request's length; the rotation tables are cut to the engine's longest context
UNIT_ALPHA = 1.702         # g * sigmoid(UNIT_ALPHA * g) in the clamped gated unit


def _mixer(config: ZabusunConfig, layer: ZabusunLayer, positions: int) -> PartSpec:
    left, rotation = layer.left, None
    if left.rot is not None:
        scaling = None if left.rot.scaling is None else {"kind": "yarn", **dict(left.rot.scaling)}
        rotation = PartSpec("rope", {"head_dim": left.dim, "theta": left.rot.base, "max_positions": positions, "rotary_dim": left.rot.dims,
                                     "scaling": scaling, "layout": "halves"})
    attention = PartSpec("gqa_attention", {
        "width": config.width, "n_heads": left.heads, "n_kv_heads": left.kv_heads, "head_dim": left.dim, "value_dim": left.vdim,
        "scale": left.scale, "position": rotation, "qk_norm_eps": config.norm_eps, "weighting": "sigmoid", "score_bias": True, "head_gate": True,
        "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "score_bias": "pb", "head_gate": "g"},
    })
    recurrent = PartSpec("min_gru", {"width": config.width, "channels": layer.right_width})
    return PartSpec("weighted_mixers", {"mixers": (attention, recurrent), "prefixes": ("left.", "right."), "scales": (layer.left_scale, layer.right_scale)})


def _feed_forward(config: ZabusunConfig, layer: ZabusunLayer) -> Optional[PartSpec]:
    mlp = layer.mlp
    if mlp is None:
        return None
    if mlp.kind == "dense":
        return PartSpec("clamped_glu", {"width": config.width, "intermediate": mlp.ff, "limit": mlp.limit, "alpha": UNIT_ALPHA,
                                        "names": {"gate": "gate", "up": "up", "down": "down"}})
    return PartSpec("expert_mixture", {
        "width": config.width, "intermediate": mlp.ff, "experts": mlp.experts, "top": mlp.top, "activation": "clamped", "limit": mlp.limit,
        "alpha": UNIT_ALPHA, "routing": "sigmoid", "share_normalized": False, "weigh": "input",
    })


def zabusun_spec(config: ZabusunConfig, max_positions: Optional[int] = None) -> ModelSpec:
    positions = MAX_POSITIONS if max_positions is None else int(max_positions)
    norm = PartSpec("rmsnorm", {"width": config.width, "eps": config.norm_eps, "weight_name": ""})
    layers = []
    for index, layer in enumerate(config.layers):
        feed_forward = _feed_forward(config, layer)
        layers.append(LayerSpec(f"l{index}.", PartSpec("output_norm", {
            "mixer": _mixer(config, layer, positions), "feed_forward": feed_forward, "mixer_norm": norm, "ffn_norm": None if feed_forward is None else norm,
        })))
    return ModelSpec(
        width=config.width,
        vocab_size=config.vocab,
        max_positions=positions,
        embedding_name="embed",
        lm_head_name=None,
        final_norm=norm,
        final_norm_prefix="final.norm",
        layers=tuple(layers),
        order=tuple(RunSpec(index) for index in range(len(config.layers))),
        eos_token_ids=config.eos_token_ids,
        logit_scale=config.logit_scale,
        embedding_norm=norm,
        embedding_norm_prefix="embed.norm",
    )
