"""A plain, slow statement of the Zabusun design, one function per mechanism.

Everything here is written from the equations alone, token by token where the design is
sequential, on the CPU, in one dtype (float64 by default); it shares no code with
``pylon_b200``.  A model is a dict ``config`` (the keys of ``config.json``) and a dict
``weights`` (tensor name -> ``torch.Tensor``).

Notation: ``h`` is a ``[T, width]`` block of one sequence, ``T`` tokens from position 0.
"""
from __future__ import annotations

import math
from typing import Mapping, Optional

import torch


# ---------------------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------------------
def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last dimension (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def sigmoid(x: torch.Tensor) -> torch.Tensor:
    """Without overflow on either side."""
    small = torch.exp(-x.abs())
    return torch.where(x >= 0, 1.0 / (1.0 + small), small / (1.0 + small))


def embed(tokens: list[int], w: Mapping[str, torch.Tensor], eps: float) -> torch.Tensor:
    """The stream a sequence starts with: the tokens' rows of the table, normed."""
    return rms_unit(w["embed"][torch.tensor(tokens)], eps) * w["embed.norm"]


def add_normed(x: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """A sublayer's output joins the stream: the norm stands on the output, the stream itself is never normed."""
    return x + rms_unit(y, eps) * weight


# ---------------------------------------------------------------------------------------
# rotation
# ---------------------------------------------------------------------------------------
def rotary_frequencies(dims: int, base: float, scaling: Optional[Mapping[str, float]]) -> tuple[torch.Tensor, float]:
    """float64 frequencies of the ``dims / 2`` pairs and the factor on cos and sin (YaRN when ``scaling`` is given)."""
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    if scaling is None:
        return freq, 1.0
    factor, original = scaling["factor"], scaling["original"]
    pair_of = [dims * math.log(original / (2.0 * math.pi * scaling[key])) / (2.0 * math.log(base)) for key in ("fast", "slow")]
    lo, hi = max(math.floor(pair_of[0]), 0), min(math.ceil(pair_of[1]), dims - 1)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        freq[i] = freq[i] / factor * ramp + freq[i] * (1.0 - ramp)
    return freq, 0.1 * math.log(factor) + 1.0


def rotate_halves(x: torch.Tensor, freq: torch.Tensor, gain: float) -> torch.Tensor:
    """``x [T, heads, dim]``: rotates the first ``2 len(freq)`` elements of every head by the token's position, element i with
    element i + len(freq)."""
    half = freq.shape[0]
    angle = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * freq
    cos, sin = (torch.cos(angle) * gain).to(x.dtype)[:, None], (torch.sin(angle) * gain).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half : 2 * half]
    return torch.cat((u * cos - v * sin, v * cos + u * sin, x[..., 2 * half :]), dim=-1)


# ---------------------------------------------------------------------------------------
# the two mixers side by side
# ---------------------------------------------------------------------------------------
def sigmoid_attention(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    """Grouped-query attention whose weights are ``sigmoid(score + pb)``, nothing divided by their sum; heads gated."""
    heads, kv_heads, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    count = h.shape[0]
    q = rms_unit((h @ w[p + "q"].T).view(count, heads, dim), eps) * w[p + "q.norm"]
    k = rms_unit((h @ w[p + "k"].T).view(count, kv_heads, dim), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(count, kv_heads, vdim)
    rot = m.get("rot")
    if rot is not None:
        freq, gain = rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q, k = rotate_halves(q, freq, gain), rotate_halves(k, freq, gain)
    gate = sigmoid(h @ w[p + "g"].T)
    out = torch.zeros(count, heads, vdim, dtype=h.dtype)
    for t in range(count):
        for head in range(heads):
            g = head // (heads // kv_heads)
            weights = sigmoid((k[: t + 1, g] @ q[t, head]) * m["scale"] + w[p + "pb"][head])
            out[t, head] = (weights @ v[: t + 1, g]) * gate[t, head]
    return out.view(count, heads * vdim) @ w[p + "o"].T


def min_gru(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str) -> torch.Tensor:
    """The gated recurrence whose gates read the current token only, from a state of zeros."""
    z = sigmoid(h @ w[p + "z"].T + w[p + "z.b"])
    u = h @ w[p + "x"].T + w[p + "x.b"]
    candidate = torch.where(u >= 0, u + 0.5, sigmoid(u))
    g = h @ w[p + "g"].T
    state = torch.zeros(u.shape[1], dtype=h.dtype)
    read = []
    for t in range(h.shape[0]):
        state = (1.0 - z[t]) * state + z[t] * candidate[t]
        read.append(state * (g[t] * sigmoid(g[t])))
    return torch.stack(read) @ w[p + "o"].T


def mixer(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    return m["left_scale"] * sigmoid_attention(h, w, p + "left.", m["left"], eps) + m["right_scale"] * min_gru(h, w, p + "right.")


# ---------------------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------------------
def clamped_unit(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def experts(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, mlp: Mapping) -> torch.Tensor:
    """Every token through the ``top`` experts with the largest sigmoid scores; an expert reads the token times its score."""
    scores = sigmoid(h @ w[p + "router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(mlp["router"]["experts"]), key=lambda e: (-float(scores[t, e]), e))
        for e in order[: mlp["router"]["top"]]:
            out[t] += clamped_unit((scores[t, e] * h[t])[None], w, f"{p}e{e}.", mlp["expert"]["limit"])[0]
    return out


def feed_forward(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, mlp: Mapping) -> torch.Tensor:
    return clamped_unit(h, w, p, mlp["limit"]) if mlp["kind"] == "dense" else experts(h, w, p, mlp)


# ---------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------
def forward(config: Mapping, weights: Mapping[str, torch.Tensor], tokens: list[int], dtype: torch.dtype = torch.float64,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence from position 0; ``layers_out`` receives the stream after every layer."""
    w = {name: tensor.to(dtype) for name, tensor in weights.items()}
    eps = config["norm"]["eps"]
    x = embed(tokens, w, eps)
    for index, layer in enumerate(config["layers"]):
        p = f"l{index}."
        x = add_normed(x, mixer(x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = add_normed(x, feed_forward(x, w, p + "mlp.", layer["mlp"]), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms_unit(x, eps) * w["final.norm"]) @ w["embed"].T * config["logit_scale"]
