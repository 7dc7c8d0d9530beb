"""Small Nadilorn-shaped models with random weights for the tests, and the comparison they share."""
from __future__ import annotations

import math

import torch

from bamudra_case import error, tokens  # noqa: F401
from oracle import nadilorn_oracle
from tilemega_b200.registry import tensor_shapes


def layer(heads, kv_heads, dim, vdim, rot, window, mlp=None, base=10000.0, factor=2.5, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                                           "rot": {"base": base, "dims": rot, "scaling": {"factor": factor}},
                                           "scale": dim ** -0.5 if scale is None else scale}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def model(width, vocab, layers, eps=1e-5):
    return {"architecture": "Nadilorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


CASES = {
    # nothing a multiple of anything, unequal layers, one without a feed-forward
    "odd": model(86, 203, [layer(9, 3, 20, 28, 12, 19, moe(7, 3, 50)), layer(4, 1, 36, 10, 36, 33, dense(70), base=300.0, factor=1.5),
                           layer(3, 3, 18, 18, 2, 50), layer(2, 1, 12, 14, 6, 27, moe(5, 2, 21), factor=4.0)], eps=1e-3),
    # equal sizes everywhere, unscaled angles, every expert used by every token
    "even": model(128, 256, [layer(4, 4, 32, 32, 32, 24, moe(4, 4, 128), factor=1.0), layer(4, 4, 32, 32, 32, 24, dense(128), factor=1.0)]),
    # ones: a head, an expert, a window of one position, values one wide (sublayers of rank 1 would leave the norm behind them
    # nothing but a sign, which rounding decides where it is close)
    "ones": model(24, 31, [layer(1, 1, 8, 12, 2, 1, moe(1, 1, 24)), layer(10, 10, 2, 1, 2, 5, moe(3, 1, 17)), layer(12, 6, 8, 1, 4, 3, dense(15))]),
    # large heads, values wider and narrower than keys, many experts
    "wide": model(264, 515, [layer(4, 1, 256, 168, 64, 70, moe(40, 8, 72)), layer(2, 2, 104, 256, 104, 130, dense(300)),
                             layer(2, 1, 200, 40, 128, 300, moe(33, 1, 16))]),
    # many query heads per key head
    "grouped": model(96, 128, [layer(34, 2, 16, 24, 8, 45, moe(9, 2, 48)), layer(20, 1, 48, 32, 24, 300, dense(40))]),
}


def weights(config, seed=0, coded=False):
    """bf16-representable fp32 tensors of unit-sized activations: matrices N(0, 1/columns), norm weights around 1.

    `coded`: which experts a token takes is made to rest on no close call. As many of the first columns as a layer has
    experts at most hold a token's own permutation of evenly spaced levels, no norm adds to these columns, and an
    expert's logit is one of them, give or take a little of the rest of the row."""
    generator = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, shape in tensor_shapes(config).items():
        draw = torch.randn(shape, generator=generator)
        if len(shape) == 2:
            draw = draw if name == "embed" else draw / math.sqrt(shape[1])
        else:
            draw = 1.0 + 0.1 * draw
        tensors[name] = draw
    counts = {f"l{index}.": item["mlp"]["router"]["experts"] for index, item in enumerate(config["layers"])
              if item["mlp"] and item["mlp"]["kind"] == "moe"}
    if coded and counts:
        most = max(counts.values())
        levels = torch.linspace(-2.0, 2.0, most)
        for token in range(config["vocab"]):
            tensors["embed"][token, :most] = levels[torch.randperm(most, generator=generator)]
        for index in range(len(config["layers"])):
            for norm in ("norm1", "norm2"):
                if f"l{index}.{norm}" in tensors:
                    tensors[f"l{index}.{norm}"][:most] = 0.0
        for prefix, count in counts.items():
            router = tensors[prefix + "mlp.router"]
            router *= 0.01
            router[:, :most] = 0.0
            router[torch.arange(count), torch.randperm(most, generator=generator)[:count]] = 1.0
    return {name: tensor.to(torch.bfloat16).float() for name, tensor in tensors.items()}


def weights_for(config, dtype, seed=0):
    """In 32 bits any router will do; in bf16 the choice of experts must not hang on rounding."""
    return weights(config, seed, coded=dtype == "bf16")


def truth(config, tensors, ids):
    """(logits, residual stream per layer) in float64, as fp32."""
    logits, kept = nadilorn_oracle.forward(config, tensors, ids, torch.float64)
    return logits.float(), kept.float()


TOLERANCE = {"f32": 3e-5, "bf16": 0.06}
