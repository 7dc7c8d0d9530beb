"""Small Mozidra-shaped models with random weights for the tests, and the comparison they share."""
from __future__ import annotations

import math

import torch

from bamudra_case import error, tokens  # noqa: F401
from oracle import mozidra_oracle
from tilemega_b200.registry import tensor_shapes


def latent(heads, dim, vdim, rank, window, mlp=None, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
                                                  "scale": dim ** -0.5 if scale is None else scale}, "mlp": mlp}


def grouped(heads, kv_heads, dim, vdim, rot, window, mlp=None, base=10000.0, scale=None, mixing=True):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                                           "rot": {"base": base, "dims": rot}, "scale": dim ** -0.5 if scale is None else scale, "v_mix": mixing},
            "mlp": mlp}


def moe(experts, top, ff, groups=1, keep=1, shared=24, limit=1.5, shared_limit=0.8):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}},
            "expert": {"ff": ff, "limit": limit}, "shared": {"ff": shared, "limit": shared_limit}}


def model(width, vocab, layers, streams=2, eps=1e-5):
    return {"architecture": "Mozidra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "streams": streams, "layers": layers}


CASES = {
    # nothing a multiple of anything, unequal layers, some without a feed-forward, one whose values are not mixed
    "odd": model(86, 203, [latent(5, 20, 28, 43, 19, moe(9, 3, 50, 3, 2, shared=70)), grouped(9, 3, 20, 28, 12, 19, moe(6, 2, 21, 2, 1, limit=0.7)),
                           grouped(4, 2, 18, 10, 18, 33, mixing=False), latent(3, 36, 10, 27, 50), grouped(6, 6, 22, 14, 8, 40, moe(10, 4, 33, 5, 3), base=300.0),
                           latent(7, 12, 30, 90, 24, moe(4, 1, 40, 4, 4, shared=9))], streams=3, eps=1e-3),
    # equal sizes everywhere, every expert used by every token, one group, attention layers first and last
    "even": model(128, 256, [grouped(4, 4, 32, 32, 32, 24, moe(4, 4, 128, shared=128)), latent(4, 32, 32, 32, 24, moe(4, 4, 128, shared=128)),
                             grouped(4, 4, 32, 32, 32, 24, moe(4, 4, 128, shared=128))], streams=4),
    # ones: a stream, a head, an expert, a window of one position, values one wide, a latent row of one column
    "ones": model(24, 31, [latent(1, 8, 12, 1, 1, moe(1, 1, 24)), grouped(10, 10, 2, 1, 2, 5, moe(3, 1, 17, 3, 1, shared=1)), latent(12, 1, 1, 9, 3),
                           grouped(5, 5, 4, 2, 2, 7, moe(2, 1, 1))], streams=1),
    # large heads, values wider and narrower than keys, many experts in many groups, a wide latent row
    "wide": model(264, 515, [latent(4, 200, 72, 300, 70, moe(40, 8, 72, 10, 4)), grouped(2, 2, 104, 256, 104, 130, moe(33, 1, 16, 11, 2)),
                             latent(2, 64, 256, 512, 300, moe(36, 6, 40, 4, 1)), grouped(4, 2, 256, 256, 64, 90)], streams=5),
    # many heads on a latent row and per key head
    "crowd": model(96, 128, [latent(70, 16, 24, 140, 45, moe(9, 2, 48, 3, 2)), latent(20, 24, 8, 64, 300), grouped(34, 2, 16, 24, 8, 45, moe(8, 3, 20, 2, 2)),
                             grouped(20, 1, 48, 48, 24, 300), latent(33, 8, 16, 250, 37)], streams=2),
    # latent rows wider than the tiles, windows over everything
    "vast": model(64, 90, [latent(3, 16, 12, 600, None, moe(4, 2, 24, 2, 1)), grouped(4, 2, 16, 16, 16, None), latent(2, 24, 24, 1024, 40)], streams=2),
}


def weights(config, seed=0, coded=False):
    """bf16-representable fp32 tensors of unit-sized activations: matrices N(0, 1/columns), norm factors around 1, streams
    mixed a little.

    `coded`: which experts a token takes is made to rest on no close call. As many of the first columns as a layer has
    experts at most hold a token's own permutation of evenly spaced levels, no sublayer adds to these columns, an expert's
    logit is one of them, give or take a little of the rest of the row, and a correction lifts or sinks an expert by more
    than scores differ."""
    generator = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, shape in tensor_shapes(config).items():
        draw = torch.randn(shape, generator=generator)
        last = name.rsplit(".", 1)[-1]
        if ".hc" in name:
            count = shape[0]
            draw = {"in": (1 + 0.2 * draw) / count, "out": 1 + 0.2 * draw,
                    "mix": 0.7 * torch.eye(count) + (0.3 + 0.1 * draw.abs()) / count if last == "mix" else None}[last]
        elif last == "vmix":
            draw = 0.5 + 0.15 * draw
        elif last == "correction":
            draw = 0.05 * draw
        elif last == "sink":
            draw = 0.5 + draw
        elif last == "b":
            draw = 0.3 * draw
        elif len(shape) == 2:
            draw = draw if name == "embed" else draw / math.sqrt(shape[1])
        elif name.endswith((".mix.q.norm", ".mix.k.norm", ".mix.dkv.norm")):
            draw = 1.0 + 0.1 * draw
        else:
            draw = 0.1 * draw                                    # stored as the distance from one
        tensors[name] = draw
    counts = {f"l{index}.": item["mlp"]["router"]["experts"] for index, item in enumerate(config["layers"]) if item["mlp"]}
    if coded and counts:
        most = max(counts.values())
        levels = torch.linspace(-2.0, 2.0, most)
        for token in range(config["vocab"]):
            tensors["embed"][token, :most] = levels[torch.randperm(most, generator=generator)]
        for name, tensor in tensors.items():
            if name.endswith((".mix.o", ".down")):
                tensor[:most] = 0.0
            if name.endswith((".norm1", ".norm2")):
                tensor[:most] = 0.0
        for prefix, count in counts.items():
            router = tensors[prefix + "mlp.router"]
            router *= 0.01
            router[:, :most] = 0.0
            router[torch.arange(count), torch.randperm(most, generator=generator)[:count]] = 2.0
            tensors[prefix + "mlp.correction"] = 1.5 * torch.randint(-1, 2, (count,), generator=generator).float()
    return {name: tensor.to(torch.bfloat16).float() for name, tensor in tensors.items()}


def weights_for(config, dtype, seed=0):
    """In 32 bits any router will do; in bf16 the choice of experts must not hang on rounding."""
    return weights(config, seed, coded=dtype == "bf16")


def truth(config, tensors, ids):
    """(logits, summed residual streams per layer) in float64, as fp32."""
    logits, kept = mozidra_oracle.forward(config, tensors, ids, torch.float64)
    return logits.float(), kept.float()


TOLERANCE = {"f32": 3e-5, "bf16": 0.06}
