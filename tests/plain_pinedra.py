"""A plain, slow statement of the Pinedra design, one function per mechanism.

Everything here is written from the equations alone, query by query, on the CPU, in one dtype (float64 by default); it
shares no code with ``pylon_b200``.  A model is a dict ``config`` (the keys of ``config.json``) and a dict ``weights``
(tensor name -> ``torch.Tensor``).

Notation: ``h`` is a ``[T, width]`` block of one sequence, ``T`` tokens from position 0.
"""
from __future__ import annotations

import math
from typing import Callable, Mapping, Optional

import torch


# ---------------------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------------------
def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last dimension (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def one_number_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose weight is one number for all coordinates."""
    return rms_unit(x, eps) * gain.reshape(())


def sigmoid(x: torch.Tensor) -> torch.Tensor:
    small = torch.exp(-x.abs())
    return torch.where(x >= 0, 1.0 / (1.0 + small), small / (1.0 + small))


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * sigmoid(x)


def query_factor(position: int, coef: float, every: float) -> float:
    """What a query at this position is multiplied by: steps up logarithmically every ``every`` positions."""
    return 1.0 + coef * math.log(math.floor((position + 1) / every) + 1.0)


def slope(head: int, heads: int) -> float:
    """What a position of distance takes off the scores of a head."""
    return 2.0 ** (-8.0 * (head + 1) / heads)


def rotate_halves(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """``x [T, heads, dim]``: rotates the first ``dims`` elements of every head by the token's position, element i with
    i + dims / 2."""
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    angle = torch.arange(x.shape[0], dtype=torch.float64).unsqueeze(1) * freq
    cos, sin = torch.cos(angle).to(x.dtype).unsqueeze(1), torch.sin(angle).to(x.dtype).unsqueeze(1)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat((u * cos - v * sin, v * cos + u * sin, x[..., dims:]), dim=-1)


# ---------------------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------------------
def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, score: Callable[[int, int, torch.Tensor, torch.Tensor], torch.Tensor],
           first: Callable[[int], int] = lambda i: 0, plus_one: bool = False) -> torch.Tensor:
    """``q [T, H, d]``, ``k [T, G, d]``, ``v [T, G, e]`` -> ``[T, H * e]``.  ``score(i, head, dots, keys)`` turns the products of query i
    with the keys of positions ``keys`` into scores; ``first(i)`` is the first position that i sees; ``plus_one``: the
    softmax's denominator holds one more, a key of score zero without a value."""
    count, heads = q.shape[0], q.shape[1]
    per = heads // k.shape[1]
    rows = []
    for i in range(count):
        keys = torch.arange(first(i), i + 1)
        out = []
        for head in range(heads):
            s = score(i, head, k[keys, head // per] @ q[i, head], keys)
            top = s.max()
            if plus_one:
                top = torch.clamp(top, min=0.0)
            e = torch.exp(s - top)
            total = e.sum() + (torch.exp(-top) if plus_one else 0.0)
            out.append((e / total) @ v[keys, head // per])
        rows.append(torch.cat(out))
    return torch.stack(rows)


def shared_value_attention(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    """'attention': the values are the projected keys as they are before their norm; q and k are normed over their whole rows;
    biases on q, k and the output; every output element gated."""
    heads, kv_heads, dim = m["heads"], m["kv_heads"], m["dim"]
    q = h @ w[p + "q"].T + w[p + "q.b"]
    k = h @ w[p + "k"].T + w[p + "k.b"]
    v = k.view(-1, kv_heads, dim)
    q = (rms_unit(q, eps) * w[p + "q.norm"]).view(-1, heads, dim)
    k = (rms_unit(k, eps) * w[p + "k.norm"]).view(-1, kv_heads, dim)
    out = attend(q, k, v, lambda i, head, dots, keys: dots * m["scale"])
    return (out * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T + w[p + "o.b"]


def sloped_attention(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    """'attention_2': q and k normed per head, queries times a factor that grows with their position, a slope per head on the
    distance, one added to the softmax's denominator; every output element gated."""
    heads, kv_heads, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit((h @ w[p + "q"].T).view(-1, heads, dim), eps) * w[p + "q.norm"]
    k = rms_unit((h @ w[p + "k"].T).view(-1, kv_heads, dim), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(-1, kv_heads, vdim)
    if m.get("q_temp") is not None:
        factors = torch.tensor([query_factor(i, m["q_temp"]["coef"], m["q_temp"]["every"]) for i in range(h.shape[0])], dtype=h.dtype)
        q = q * factors.view(-1, 1, 1)
    out = attend(q, k, v, lambda i, head, dots, keys: dots * m["scale"] - slope(head, heads) * (i - keys).to(dots.dtype), plus_one=True)
    return (out * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def chunk_attention(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    """'attention_3': biases on q, k, v; part of every head rotated; soft-capped scores inside chunks of positions; every head gated."""
    heads, kv_heads, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(-1, heads, dim)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(-1, kv_heads, dim)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(-1, kv_heads, vdim)
    if m.get("rot") is not None:
        q, k = rotate_halves(q, m["rot"]["dims"], m["rot"]["base"]), rotate_halves(k, m["rot"]["dims"], m["rot"]["base"])
    cap, mask = m.get("softcap"), m.get("mask")

    def score(i, head, dots, keys):
        s = dots * m["scale"]
        return s if cap is None else cap * torch.tanh(s / cap)

    out = attend(q, k, v, score, first=(lambda i: 0) if mask is None else (lambda i: i // mask["size"] * mask["size"]))
    gate = sigmoid(h @ w[p + "g"].T)
    return (out.view(-1, heads, vdim) * gate.unsqueeze(-1)).reshape(out.shape) @ w[p + "o"].T


MIXERS = {"attention": shared_value_attention, "attention_2": sloped_attention, "attention_3": chunk_attention}


# ---------------------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------------------
def unit(x: torch.Tensor, w: Mapping[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def choose(scores: torch.Tensor, correction: torch.Tensor, top: int, groups: Optional[Mapping]) -> list[int]:
    """Which of one token's experts are used: the ``top`` largest of score + correction, among the groups whose largest such number is largest."""
    value = (scores + correction).tolist()
    allowed = list(range(len(value)))
    if groups is not None:
        size = len(value) // groups["count"]
        worth = [max(value[g * size:(g + 1) * size]) for g in range(groups["count"])]
        best = sorted(range(len(worth)), key=lambda g: -worth[g])[: groups["keep"]]
        allowed = [e for e in allowed if e // size in best]
    return sorted(allowed, key=lambda e: -value[e])[:top]


def mixture(h: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping) -> torch.Tensor:
    """Experts chosen by softmax scores with a correction, weighted by the plain scores times a factor; the router's last outputs
    are experts that hand their input back; one expert more for every token."""
    router = m["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        scores = torch.softmax(w[p + "router"] @ h[t], dim=0)
        for e in choose(scores, w[p + "correction"], router["top"], router.get("groups")):
            y = unit(h[t], w, f"{p}e{e}.") if e < router["experts"] else h[t]
            out[t] += scores[e] * router["scale"] * y
    if m.get("shared") is not None:
        out = out + unit(h, w, p + "shared.")
    return out


# ---------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------
def run_order(config: Mapping) -> list[tuple[int, bool]]:
    """(layer, whether the embedding output is added right before it) of every layer run."""
    count = len(config["layers"])
    loop = config.get("loop")
    if loop is None:
        return [(i, False) for i in range(count)]
    order = [(i, False) for i in range(loop["start"])]
    for turn in range(loop["times"]):
        order += [(i, turn > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], count)]


def layer(x: torch.Tensor, w: Mapping[str, torch.Tensor], index: int, spec: Mapping, eps: float) -> torch.Tensor:
    h = one_number_norm(x, w[f"l{index}.norm1"], eps)
    y = MIXERS[spec["type"]](h, w, f"l{index}.mix.", spec["mixer"], eps)
    if spec.get("mlp") is not None:
        y = y + mixture(h, w, f"l{index}.mlp.", spec["mlp"])
    return x + y


def forward(config: Mapping, weights: Mapping[str, torch.Tensor], tokens: list[int], dtype: torch.dtype = torch.float64,
            taps: Optional[list] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence; ``taps`` receives the stream after every layer run."""
    w = {name: tensor.to(dtype) for name, tensor in weights.items()}
    eps = config["norm"]["eps"]
    embedded = w["embed"][torch.tensor(tokens)] * config["embedding"]["scale"]
    x = embedded
    for index, again in run_order(config):
        if again:
            x = x + embedded
        x = layer(x, w, index, config["layers"][index], eps)
        if taps is not None:
            taps.append(x.clone())
    return one_number_norm(x, w["final.norm"], eps) @ w["head"].T
