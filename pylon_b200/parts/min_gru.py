"""A minimal gated recurrence over channels (minGRU): a gated unit whose gate and candidate read the current token only, so that the
state enters linearly and a row of tokens can be walked in pieces side by side.

Per token, with h the layer's input and C channels:

* ``z = sigmoid(W_z h + b_z)``, ``u = W_x h + b_x``; the candidate is ``u + 1/2`` where ``u >= 0`` and ``sigmoid(u)`` where ``u < 0`` (positive and
  continuous);
* ``S = (1 - z) S + z * candidate`` from ``S = 0``;
* the output projection of ``S * silu(W_g h)``.

What a request carries from token to token is S, one float32 state slot of C numbers.  The three projections are one product; everything
behind them is float32 (``csrc/min_gru.cu``).  Tensors: ``z``, ``x``, ``g`` ``[C, width]``, ``z.b``, ``x.b`` ``[C]``, ``o [width, C]``.
"""
from __future__ import annotations

from typing import Mapping, Optional, Sequence

import torch

from pylon_b200.kernels import ops
from pylon_b200.parts.base import MIXERS, CacheNeed, LayerCache, Mixer, StateNeed, StepView, TensorDecl


@MIXERS.register("min_gru")
class MinGRU(Mixer):
    takes_padding = True    # the kernels walk rows, and skip rows without tokens
    splits_products = True

    def __init__(self, width: int, channels: int, names: Optional[Mapping[str, str]] = None) -> None:
        self.width, self.channels = int(width), int(channels)
        if min(self.width, self.channels) < 1:
            raise ValueError(f"{channels} channels over a width of {width}")
        self.names = {"z": "z", "x": "x", "g": "g", "o": "o", "bias_suffix": ".b", **(names or {})}
        self.bias: Optional[torch.Tensor] = None    # float32 [2, C]: the gate's, the candidate's

    def tensors(self) -> Sequence[TensorDecl]:
        n, b = self.names, self.names["bias_suffix"]
        return [
            TensorDecl(n["z"], (self.channels, self.width)), TensorDecl(n["z"] + b, (self.channels,), "vector", (-3.0, 2.0)),
            TensorDecl(n["x"], (self.channels, self.width)), TensorDecl(n["x"] + b, (self.channels,), "vector", (0.0, 0.5)),
            TensorDecl(n["g"], (self.channels, self.width)), TensorDecl(n["o"], (self.width, self.channels)),
        ]

    def load(self, tensors: Mapping[str, torch.Tensor], dtype: torch.dtype, device: torch.device) -> None:
        n, b = self.names, self.names["bias_suffix"]
        self.input_rows = torch.cat((tensors[n["z"]], tensors[n["x"]], tensors[n["g"]]), dim=0).contiguous()   # one product: columns [z | x | g]
        self.bias = torch.stack((tensors[n["z"] + b], tensors[n["x"] + b])).contiguous()
        self.output_columns = tensors[n["o"]].contiguous()

    def weight_bytes(self) -> int:
        return (self.input_rows.numel() + self.output_columns.numel()) * self.output_columns.element_size() + 8 * self.channels

    def cache_need(self) -> CacheNeed:
        return CacheNeed(state=StateNeed((self.channels,)))

    def forward(self, h: torch.Tensor, step: StepView, cache: LayerCache) -> torch.Tensor:
        read = torch.empty((h.shape[0], self.channels), dtype=h.dtype, device=h.device)
        self.middle(ops.linear_stacked(h, self.input_rows), step, cache, read, 1.0)
        return ops.linear_for_residual(read, self.output_columns)

    def middle(self, proj: torch.Tensor, step: StepView, cache: LayerCache, out: torch.Tensor, factor: float) -> None:
        ops.min_gru(proj, self.bias, cache.state, step.q_start, step.slots, step.num_rows, step.max_q, out, factor)
