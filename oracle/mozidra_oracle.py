"""Plain, slow forward of a Mozidra-shaped decoder: one function per mechanism, whole sequences, one precision.

Test infrastructure only. Nothing here is shared with the product path: masks are built entry by entry from their
definition, latent keys and values are expanded per head, experts run token by token, angles are taken in float64.
`dtype` is the arithmetic type of everything else (float32 or float64).

Notation: X [streams, T, width] are the residual streams; what a sublayer reads is a weighted sum of them, normalised. p is
the position of a token.
"""
from __future__ import annotations

import math

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """An RMS norm whose stored weights say how far the factors are from one."""
    return rms(x, eps) * (1.0 + weight)


def collect(streams: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """What a sublayer reads: the streams' weighted sum."""
    return sum(weight[s] * streams[s] for s in range(streams.shape[0]))


def distribute(streams: torch.Tensor, mix: torch.Tensor, out: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """Every new stream t: all old streams s, each by mix[s, t], and the sublayer's output by out[t]."""
    count = streams.shape[0]
    return torch.stack([sum(mix[s, t] * streams[s] for s in range(count)) + out[t] * y for t in range(count)])


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """Rotary positions on the first `dims` entries of the last axis of x [T, heads, dim]: neighbours 2i and 2i + 1 turn
    by the angle p * base^(-2i/dims)."""
    out = x.clone()
    for i in range(dims // 2):
        angle = positions.double() * base ** (-2.0 * i / dims)
        cos, sin = angle.cos().to(x.dtype)[:, None], angle.sin().to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * cos - v * sin, v * cos + u * sin
    return out


def visible(i: int, j: int, size: int | None) -> bool:
    """Does position i see position j: the last `size` positions including itself (None: everything before)."""
    return 0 <= i - j and (size is None or i - j < size)


def softmax_with_sink(score: torch.Tensor, seen: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (exp(sink) + sum of the seen exp(s)): a softmax that may also rest on a key of score `sink` without a
    value."""
    score = score.masked_fill(~seen, -math.inf)
    top = torch.maximum(score.max(-1, keepdim=True).values, sink)
    weight = torch.exp(score - top)
    return weight / (torch.exp(sink - top) + weight.sum(-1, keepdim=True))


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, size: int | None, sinks: torch.Tensor) -> torch.Tensor:
    """Grouped heads over a sliding window. q [T, heads, dim], k [T, kv_heads, dim], v [T, kv_heads, vdim], sinks [heads]."""
    steps, heads, _ = q.shape
    group = heads // k.shape[1]
    seen = torch.tensor([[visible(i, j, size) for j in range(steps)] for i in range(steps)])
    out = torch.empty(steps, heads, v.shape[-1], dtype=q.dtype)
    for head in range(heads):
        kv = head // group
        out[:, head] = softmax_with_sink((q[:, head] @ k[:, kv].T) * scale, seen, sinks[head]) @ v[:, kv]
    return out


def window_of(spec: dict) -> int | None:
    return (spec.get("mask") or {}).get("size")


def attention_mixer(h: torch.Tensor, positions: torch.Tensor, spec: dict, w, eps: float, first_values: torch.Tensor | None):
    """(mixer output, the layer's own values before mixing [T, kv_heads * vdim])."""
    heads, groups = spec["heads"], spec["kv_heads"]
    q = rms(h @ w("q").T + w("q.b"), eps) * w("q.norm")         # one mean over all heads together
    k = rms(h @ w("k").T + w("k.b"), eps) * w("k.norm")
    own = h @ w("v").T + w("v.b")
    v = own
    if first_values is not None:
        v = (1.0 - w("vmix")) * own + w("vmix") * first_values
    q, k, v = q.reshape(-1, heads, spec["dim"]), k.reshape(-1, groups, spec["dim"]), v.reshape(-1, groups, spec["vdim"])
    rot = spec.get("rot")
    if rot:
        q, k = rotate_pairs(q, positions, rot["base"], rot["dims"]), rotate_pairs(k, positions, rot["base"], rot["dims"])
    o = attend(q, k, v, spec["scale"], window_of(spec), w("sink"))
    return o.reshape(h.shape[0], -1) @ w("o").T, own


def latent_mixer(h: torch.Tensor, spec: dict, w, eps: float) -> torch.Tensor:
    """Attention whose keys and values are two linear images, per head, of one normalised latent row per token."""
    heads = spec["heads"]
    q = (h @ w("q").T).reshape(-1, heads, spec["dim"])
    c = rms(h @ w("dkv").T, eps) * w("dkv.norm")
    k = (c @ w("uk").T).reshape(-1, heads, spec["dim"])
    v = (c @ w("uv").T).reshape(-1, heads, spec["vdim"])
    o = attend(q, k, v, spec["scale"], window_of(spec), w("sink"))
    return o.reshape(h.shape[0], -1) @ w("o").T


def clipped_unit(h: torch.Tensor, limit: float, w) -> torch.Tensor:
    g = (h @ w("gate").T).clamp(max=limit)
    u = (h @ w("up").T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w("down").T


def route(z: torch.Tensor, correction: torch.Tensor, top: int, groups: int, keep: int) -> tuple[list[int], list[float]]:
    """One token's experts and their weights from its logits z. Scores are a softmax; experts are ranked by score plus
    correction, inside the `keep` groups of neighbours whose best such rank is largest; weights are the scores themselves
    over their sum."""
    score = torch.softmax(z, dim=-1)
    rank = (score + correction).tolist()
    size = len(rank) // groups
    best = sorted(range(groups), key=lambda g: (-max(rank[g * size:(g + 1) * size]), g))[:keep]
    open_experts = [e for e in range(len(rank)) if e // size in best]
    chosen = sorted(open_experts, key=lambda e: (-rank[e], e))[:top]
    total = sum(score[e] for e in chosen) + 1e-20
    return chosen, [score[e] / total for e in chosen]


def expert_mixture(h: torch.Tensor, spec: dict, w) -> torch.Tensor:
    router = spec["router"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    z = h @ w("router").T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for expert, weight in zip(*route(z[t], w("correction"), router["top"], groups["count"], groups["keep"])):
            out[t] += weight * clipped_unit(h[t], spec["expert"]["limit"], lambda name: w(f"e{expert}.{name}"))
    if spec.get("shared"):
        open_by = torch.sigmoid(h @ w("shared.sg").T)
        out = out + open_by * clipped_unit(h, spec["shared"]["limit"], lambda name: w("shared." + name))
    return out


def forward(config: dict, tensors: dict[str, torch.Tensor], tokens: list[int], dtype: torch.dtype = torch.float32):
    """(logits [T, vocab], sum of the residual streams after every layer [layers, T, width]) of one whole sequence."""
    cast: dict[str, torch.Tensor] = {}

    def get(name: str) -> torch.Tensor:
        if name not in cast:
            cast[name] = tensors[name].to(dtype)
        return cast[name]

    eps = config["norm"]["eps"]
    positions = torch.arange(len(tokens))
    x = get("embed")[torch.tensor(tokens, dtype=torch.long)]
    streams = torch.stack([x] * config["streams"])
    first_values, kept = None, []
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{index}."
        mix = lambda name: get(prefix + "mix." + name)

        def sublayer(streams, number, run):
            hyper = f"{prefix}hc{number}."
            h = centred_norm(collect(streams, get(hyper + "in")), get(f"{prefix}norm{number}"), eps)
            return distribute(streams, get(hyper + "mix"), get(hyper + "out"), run(h))

        def mixer(h):
            nonlocal first_values
            if layer["type"] == "latent_attention":
                return latent_mixer(h, layer["mixer"], mix, eps)
            mixing = layer["mixer"].get("v_mix")
            out, own = attention_mixer(h, positions, layer["mixer"], mix, eps, first_values if mixing else None)
            if mixing and first_values is None:
                first_values = own
            return out

        streams = sublayer(streams, 1, mixer)
        if layer["mlp"] is not None:
            streams = sublayer(streams, 2, lambda h: expert_mixture(h, layer["mlp"], lambda name: get(prefix + "mlp." + name)))
        kept.append(streams.sum(0))
    return centred_norm(streams.sum(0), get("final.norm"), eps) @ get("head").T, torch.stack(kept)
