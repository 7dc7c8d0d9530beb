"""Plain, slow forward of a Benarax-shaped decoder: one function per mechanism, whole sequences, one precision.

Test infrastructure only. Nothing here is shared with the product path: the recurrence runs token by token, convolutions
tap by tap, latent keys and values are expanded per head, experts run token by token, angles are taken in float64.
`dtype` is the arithmetic type of everything else (float32 or float64).

Notation: x [T, width] is the residual stream, p the position of a token, m the factor of everything added to x.
"""
from __future__ import annotations

import math

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x: torch.Tensor, weight: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """Every one of `groups` equal runs of columns over its own root mean square, then the weights."""
    parts = [rms(part, eps) for part in x.chunk(groups, dim=-1)]
    return torch.cat(parts, dim=-1) * weight


def short_convolution(h: torch.Tensor, kernel: torch.Tensor) -> torch.Tensor:
    """Causal, channel by channel: kernel [width, taps], its last tap on the token itself; zeros before the start."""
    steps, taps = h.shape[0], kernel.shape[1]
    out = torch.zeros_like(h)
    for t in range(steps):
        for back in range(min(taps, t + 1)):
            out[t] += kernel[:, taps - 1 - back] * h[t - back]
    return out


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot: dict) -> tuple[list[float], float]:
    """(angle per position of every pair, factor of cosine and sine). With `scaling`, slow pairs turn `factor` times
    slower, fast ones as before, those between by a ramp over the pair's index; cosine and sine grow a little."""
    base, dims, scaling = rot["base"], rot["dims"], rot.get("scaling")
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return plain, 1.0

    def index(turns: float) -> float:            # (real-valued) pair that turns so often over the original length
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(index(scaling["fast"])), 0)
    high = min(math.ceil(index(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x: torch.Tensor, positions: torch.Tensor, rot: dict, neighbours: bool) -> torch.Tensor:
    """Rotary positions on the last axis of x [T, heads, dims]: entries 2i and 2i + 1 turn together, or i and i + dims / 2."""
    dims = rot["dims"]
    turn, size = frequencies(rot)
    out = x.clone()
    for i, f in enumerate(turn):
        first, second = (2 * i, 2 * i + 1) if neighbours else (i, i + dims // 2)
        angle = positions.double() * f
        cos, sin = (size * angle.cos()).to(x.dtype)[:, None], (size * angle.sin()).to(x.dtype)[:, None]
        u, v = x[..., first], x[..., second]
        out[..., first], out[..., second] = u * cos - v * sin, v * cos + u * sin
    return out


def causal_softmax(score: torch.Tensor) -> torch.Tensor:
    """score [T, T]: row i over the keys j <= i."""
    places = torch.arange(score.shape[0])
    return torch.softmax(score.masked_fill(places[None, :] > places[:, None], -math.inf), dim=-1)


def latent_mixer(h: torch.Tensor, positions: torch.Tensor, spec: dict, w, eps: float, neighbours: bool) -> torch.Tensor:
    """Attention from queries made of a normed latent, to keys and values made of another one and a rotated key part that
    all heads share."""
    heads, dim, turned, rank, steps = spec["heads"], spec["dim"], spec["rot_dim"], spec["kv_rank"], h.shape[0]
    q = ((rms(h @ w("dq").T, eps) * w("dq.norm")) @ w("uq").T).reshape(steps, heads, dim + turned)
    down = h @ w("dkv").T
    c = rms(down[:, :rank], eps) * w("dkv.norm")
    k = (c @ w("uk").T).reshape(steps, heads, dim)
    v = (c @ w("uv").T).reshape(steps, heads, spec["vdim"])
    q_turned = rotate(q[..., dim:], positions, spec["rot"], neighbours)
    k_turned = rotate(down[:, None, rank:], positions, spec["rot"], neighbours)[:, 0]
    out = torch.empty(steps, heads, spec["vdim"], dtype=h.dtype)
    for head in range(heads):
        score = (q[:, head, :dim] @ k[:, head].T + q_turned[:, head] @ k_turned.T) * spec["scale"]
        out[:, head] = causal_softmax(score) @ v[:, head]
    return out.reshape(steps, -1) @ w("o").T


def decay_of(z: torch.Tensor) -> torch.Tensor:
    return torch.exp(-math.exp(-0.5) * torch.sigmoid(z))


def delta_recurrence(r, k, v, w, a) -> torch.Tensor:
    """One head, all [T, dim]: S <- diag(w) S - (a u) (u^T S) + k v^T with u the unit key and both terms from the old S;
    o = S^T r."""
    steps, dim = r.shape
    state = torch.zeros(dim, v.shape[1], dtype=r.dtype)
    out = torch.empty_like(v)
    for t in range(steps):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum() + 1e-6)
        state = w[t][:, None] * state - torch.outer(a[t] * u, u @ state) + torch.outer(k[t], v[t])
        out[t] = r[t] @ state
    return out


def delta_mixer(h: torch.Tensor, spec: dict, w, eps: float) -> torch.Tensor:
    heads, steps = spec["heads"], h.shape[0]
    split = lambda x: x.reshape(steps, heads, spec["dim"])
    r, k, v = (split(h @ w(name).T) for name in ("r", "k", "v"))
    decay = split(decay_of(torch.tanh(h @ w("w1").T) @ w("w2").T + w("w0")))
    removal = split(torch.sigmoid(h @ w("a").T + w("a.b")))
    o = torch.stack([delta_recurrence(r[:, i], k[:, i], v[:, i], decay[:, i], removal[:, i]) for i in range(heads)], dim=1)
    return (rms(o, eps).reshape(steps, -1) * w("norm") * torch.sigmoid(h @ w("g").T)) @ w("o").T


def clipped_unit(h: torch.Tensor, limit: float, w) -> torch.Tensor:
    g = (h @ w("gate").T).clamp(max=limit)
    u = (h @ w("up").T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w("down").T


def route(z: torch.Tensor, top: int) -> tuple[list[int], torch.Tensor]:
    """One token's experts, those of the largest logits, and their weights: a softmax over these logits alone."""
    chosen = sorted(range(len(z)), key=lambda e: (-float(z[e]), e))[:top]
    return chosen, torch.softmax(z[torch.tensor(chosen)], dim=-1)


def expert_mixture(h: torch.Tensor, spec: dict, w) -> torch.Tensor:
    z = h @ w("router").T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for expert, weight in zip(*route(z[t], spec["router"]["top"])):
            out[t] += weight * clipped_unit(h[t], spec["expert"]["limit"], lambda name: w(f"e{expert}.{name}"))
    return out


def side_input(x: torch.Tensor, e: torch.Tensor, w, eps: float) -> torch.Tensor:
    """What a layer adds from its own part e [T, dim] of the tokens' second embedding, gated by the stream."""
    return rms((gelu_tanh(x @ w("gate").T) * e) @ w("proj").T, eps) * w("norm")


def order(config: dict) -> list[int]:
    count, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(count))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], count))


def forward(config: dict, tensors: dict[str, torch.Tensor], tokens: list[int], dtype: torch.dtype = torch.float32):
    """(logits [T, vocab], residual stream after every layer run [runs, T, width]) of one whole sequence."""
    cast: dict[str, torch.Tensor] = {}

    def get(name: str) -> torch.Tensor:
        if name not in cast:
            cast[name] = tensors[name].to(dtype)
        return cast[name]

    eps, groups, m, dim = config["norm"]["eps"], config["norm"]["groups"], config["residual_mult"], config["token_side"]["dim"]
    ids, positions = torch.tensor(tokens, dtype=torch.long), torch.arange(len(tokens))
    x, kept = get("embed")[ids] * config["embedding"]["scale"], []
    for index in order(config):
        layer, prefix = config["layers"][index], f"l{index}."
        under = lambda part: lambda name: get(prefix + part + name)
        h = grouped_norm(x, get(prefix + "norm1"), groups, eps)
        read = h + short_convolution(h, get(prefix + "canon1"))
        if layer["type"] == "general_delta":
            added = delta_mixer(read, layer["mixer"], under("mix."), eps)
        else:
            added = latent_mixer(read, positions, layer["mixer"], under("mix."), eps, layer["type"] == "latent_attention")
        if layer["mlp"] is not None:
            added = added + expert_mixture(h, layer["mlp"], under("mlp."))
        x = x + m * added
        e = get("side.embed")[ids][:, index * dim:(index + 1) * dim]
        x = x + m * side_input(x, e, under("side."), eps)
        kept.append(x)
    return grouped_norm(x, get("final.norm"), groups, eps) @ get("head").T * config["logit_scale"], torch.stack(kept)
