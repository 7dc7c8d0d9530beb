"""Plain, slow forward of a Nadilorn-shaped decoder: one function per mechanism, whole sequences, one precision.

Test infrastructure only. Nothing here is shared with the product path: masks are built entry by entry from their
definition, experts run token by token, angles are taken in float64. `dtype` is the arithmetic type of everything else
(float32 or float64).

Notation: x [T, width] is the residual stream and what every sublayer reads; a sublayer's output is normalised before it
is added. p is the position of a token.
"""
from __future__ import annotations

import math

import torch


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last axis (eps inside the root), times a weight per column."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def rotate(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int, factor: float = 1.0) -> torch.Tensor:
    """Rotary positions on the first `dims` entries of the last axis of x [T, heads, dim]: entry i turns with entry
    i + dims/2 by the angle p * base^(-2i/dims) / factor."""
    half = dims // 2
    i = torch.arange(half, dtype=torch.float64)
    angle = positions.double()[:, None] * (base ** (-2.0 * i / dims) / factor)
    cos, sin = angle.cos().to(x.dtype)[:, None, :], angle.sin().to(x.dtype)[:, None, :]
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat((u * cos - v * sin, v * cos + u * sin, rest), dim=-1)


def visible(i: int, j: int, size: int | None) -> bool:
    """Does position i see position j: the last `size` positions including itself (None: everything before)."""
    return 0 <= i - j and (size is None or i - j < size)


def softmax_with_null(score: torch.Tensor, seen: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum of the seen exp(s)): a softmax that may also rest on a null key of score 0 without a value."""
    score = score.masked_fill(~seen, -math.inf)
    top = score.max(-1, keepdim=True).values.clamp_min(0.0)
    weight = torch.exp(score - top)
    return weight / (torch.exp(-top) + weight.sum(-1, keepdim=True))


def attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, size: int | None) -> torch.Tensor:
    """Grouped heads over a sliding window. q [T, heads, dim], k [T, kv_heads, dim], v [T, kv_heads, vdim]."""
    steps, heads, _ = q.shape
    group = heads // k.shape[1]
    seen = torch.tensor([[visible(i, j, size) for j in range(steps)] for i in range(steps)])
    out = torch.empty(steps, heads, v.shape[-1], dtype=q.dtype)
    for head in range(heads):
        kv = head // group
        out[:, head] = softmax_with_null((q[:, head] @ k[:, kv].T) * scale, seen) @ v[:, kv]
    return out


def attention_mixer(x: torch.Tensor, positions: torch.Tensor, spec: dict, w, eps: float) -> torch.Tensor:
    heads, groups = spec["heads"], spec["kv_heads"]
    q = rms_norm(x @ w("q").T, w("q.norm"), eps).reshape(-1, heads, spec["dim"])     # one mean over all heads together
    k = rms_norm(x @ w("k").T, w("k.norm"), eps).reshape(-1, groups, spec["dim"])
    v = (x @ w("v").T).reshape(-1, groups, spec["vdim"])
    rot = spec.get("rot")
    if rot:
        turn = (rot["base"], rot["dims"], (rot.get("scaling") or {}).get("factor", 1.0))
        q, k = rotate(q, positions, *turn), rotate(k, positions, *turn)
    o = attention(q, k, v, spec["scale"], (spec.get("mask") or {}).get("size"))
    return (o.reshape(x.shape[0], -1) * torch.sigmoid(x @ w("g").T)) @ w("o").T


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_unit(x: torch.Tensor, w) -> torch.Tensor:
    return (gelu_tanh(x @ w("gate").T) * (x @ w("up").T)) @ w("down").T


def squared_relu(z: torch.Tensor) -> torch.Tensor:
    return z.clamp_min(0.0) ** 2


def route(x: torch.Tensor, router: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """The `top` experts of each token by sigmoid(router x), and those scores as they are: ([T, top], [T, top])."""
    scores = torch.sigmoid(x @ router.T)
    chosen = torch.topk(scores, top, dim=-1)
    return chosen.indices, chosen.values


def expert_mixture(x: torch.Tensor, spec: dict, w) -> torch.Tensor:
    """Each chosen expert runs on its token's row times its score; the outputs are summed."""
    indices, scores = route(x, w("router"), spec["router"]["top"])
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for expert, score in zip(indices[t].tolist(), scores[t]):
            out[t] += squared_relu((score * x[t]) @ w(f"e{expert}.up").T) @ w(f"e{expert}.down").T
    return out


def feed_forward(x: torch.Tensor, spec: dict, w) -> torch.Tensor:
    return gated_unit(x, w) if spec["kind"] == "dense" else expert_mixture(x, spec, w)


def forward(config: dict, tensors: dict[str, torch.Tensor], tokens: list[int], dtype: torch.dtype = torch.float32):
    """(logits [T, vocab], residual stream after every layer [layers, T, width]) of one whole sequence."""
    cast: dict[str, torch.Tensor] = {}

    def get(name: str) -> torch.Tensor:
        if name not in cast:
            cast[name] = tensors[name].to(dtype)
        return cast[name]

    eps = config["norm"]["eps"]
    positions = torch.arange(len(tokens))
    x, kept = get("embed")[torch.tensor(tokens, dtype=torch.long)], []
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{index}."
        mixed = attention_mixer(x, positions, layer["mixer"], lambda name: get(prefix + "mix." + name), eps)
        x = x + rms_norm(mixed, get(prefix + "norm1"), eps)
        if layer["mlp"] is not None:
            x = x + rms_norm(feed_forward(x, layer["mlp"], lambda name: get(prefix + "mlp." + name)), get(prefix + "norm2"), eps)
        kept.append(x)
    return rms_norm(x, get("final.norm"), eps) @ get("head").T, torch.stack(kept)
