"""Pinedra as a :class:`ModelSpec`.

The configuration lists the layers; each is a ``parallel_sublayers`` block - one RMS norm (its weight a single number) whose output both
the mixer and the feed-forward read - around a ``gqa_attention`` of one of three kinds and an ``expert_mixture``, or none.  Kind
``attention``: the values are the projected keys before their norm, q and k normed over their whole rows, biases on q, k and the output.
``attention_2``: q and k normed per head, queries times a factor by position, a slope per head on the distance, a sink of score 0.
``attention_3``: biases on q, k and v, the first elements of a head rotated in halves, a soft cap, chunks of positions.  The outputs of
the first two are gated element by element, the third's head by head.  The experts are chosen by softmax scores with a correction
inside the groups whose best choice is best, weighted by the scores times a factor; the last router outputs hand their input back; a
shared expert runs for every token.  The run order repeats the loop's span, the embedding added again before every pass but the first,
each pass with caches of its own.  Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import Optional

from pylon_b200.config.model_config import PinedraAttention, PinedraConfig, PinedraFeedForward
from pylon_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, RunSpec

MAX_POSITIONS = 1 << 20    # no learnt table limits a request's length; the tables by position are cut to the engine's longest context
SLOPE_SPAN = 8.0           # the slopes on the distance: 2^(-SLOPE_SPAN (h + 1) / heads)
SINK_SCORE = 0.0           # attention_2: the softmax's denominator holds exp(SINK_SCORE)


def _mixer(config: PinedraConfig, m: PinedraAttention, positions: int) -> PartSpec:
    params = {
        "width": config.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "scale": m.scale,
        "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "output_gate": "g"},
    }
    if m.kind == "attention":
        params.update(values_from_keys=True, qk_norm="whole", qk_norm_eps=config.norm_eps, bias=True, out_bias=True, output_gate="elements")
    elif m.kind == "attention_2":
        params.update(qk_norm_eps=config.norm_eps, distance_slopes=tuple(2.0 ** (-SLOPE_SPAN * (h + 1) / m.heads) for h in range(m.heads)),
                      fixed_sink=SINK_SCORE, output_gate="elements")
        if m.temperature is not None:
            params["query_factor"] = PartSpec("log_steps", {"coef": m.temperature[0], "every": m.temperature[1], "max_positions": positions})
    else:
        params.update(bias=True, output_gate="heads", softcap=m.softcap, chunk=m.chunk)
        if m.rot is not None:
            params["position"] = PartSpec("rope", {"head_dim": m.dim, "theta": m.rot.base, "max_positions": positions, "rotary_dim": m.rot.dims,
                                                   "exact_angles": True})
    return PartSpec("gqa_attention", params)


def _feed_forward(config: PinedraConfig, mlp: Optional[PinedraFeedForward]) -> Optional[PartSpec]:
    if mlp is None:
        return None
    return PartSpec("expert_mixture", {
        "width": config.width, "intermediate": mlp.ff, "experts": mlp.experts, "top": mlp.top, "activation": "silu", "routing": "softmax_all",
        "correction": True, "groups": mlp.groups, "groups_keep": mlp.groups_keep, "group_score": "best", "share_normalized": False,
        "share_scale": mlp.scale, "identity": mlp.identity, "always_intermediate": mlp.shared_ff,
    })


def pinedra_spec(config: PinedraConfig, max_positions: Optional[int] = None) -> ModelSpec:
    positions = MAX_POSITIONS if max_positions is None else int(max_positions)
    norm = PartSpec("rmsnorm", {"width": config.width, "eps": config.norm_eps, "weight_name": "", "one_number": True})
    layers = []
    for index, layer in enumerate(config.layers):
        block = PartSpec("parallel_sublayers", {"mixer": _mixer(config, layer.mixer, positions), "feed_forward": _feed_forward(config, layer.mlp), "norm": norm})
        layers.append(LayerSpec(f"l{index}.", block))
    return ModelSpec(
        width=config.width,
        vocab_size=config.vocab,
        max_positions=positions,
        embedding_name="embed",
        lm_head_name="head",
        final_norm=norm,
        final_norm_prefix="final.norm",
        layers=tuple(layers),
        order=tuple(RunSpec(index, add_embedding=again) for index, again in config.run_order()),
        eos_token_ids=config.eos_token_ids,
        embedding_scale=config.embedding_scale,
    )
