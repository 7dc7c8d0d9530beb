"""Small Benarax-shaped models with random weights for the tests, and the comparison they share."""
from __future__ import annotations

import math

import torch

from bamudra_case import error, tokens  # noqa: F401
from oracle import benarax_oracle
from tilemega_b200.registry import tensor_shapes


def latent(heads, dim, rot, vdim, rank, q_rank, mlp=None, base=10000.0, scale=None, neighbours=True, scaling=None):
    """`neighbours`: the kind whose neighbouring entries turn together (with a scaled rotation or without)."""
    turn = {"base": base, "dims": rot} | ({"scaling": scaling} if scaling else {})
    return {"type": "latent_attention" if neighbours else "latent_attention_2",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "rot": turn,
                      "scale": (dim + rot) ** -0.5 if scale is None else scale}, "mlp": mlp}


def stretch(factor=4.0, original=64, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def delta(heads, dim, decay_rank, mlp=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim, "decay_rank": decay_rank}, "mlp": mlp}


def moe(experts, top, ff, limit=1.5):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def model(width, vocab, layers, groups=1, taps=3, side=8, loop=None, eps=1e-5, embed_scale=1.5, residual_mult=0.8, logit_scale=0.5):
    config = {"architecture": "Benarax", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups}, "canon": {"taps": taps},
              "embedding": {"scale": embed_scale}, "residual_mult": residual_mult, "logit_scale": logit_scale, "token_side": {"dim": side},
              "layers": layers}
    if loop:
        config["loop"] = dict(zip(("start", "stop", "times"), loop))
    return config


CASES = {
    # nothing a multiple of anything, unequal layers, some without a feed-forward, three passes over the middle
    "odd": model(90, 203, [latent(5, 20, 6, 28, 43, 21, moe(9, 3, 50)), delta(3, 22, 5, moe(6, 2, 21, limit=0.7)),
                           latent(3, 36, 10, 10, 27, 50, neighbours=False, base=300.0), delta(2, 37, 11), latent(7, 12, 2, 30, 90, 9, moe(4, 1, 40), scaling=stretch())],
                 groups=3, taps=4, side=7, loop=(1, 4, 3), eps=2e-2),
    # equal sizes everywhere, every expert used by every token, one group of columns, a loop that runs once
    "even": model(128, 256, [delta(4, 32, 32, moe(4, 4, 128)), latent(4, 32, 32, 32, 32, 32, moe(4, 4, 128), neighbours=False),
                             latent(4, 32, 32, 32, 32, 32, moe(4, 4, 128), scaling=stretch(1.0)), delta(4, 32, 32, moe(4, 4, 128))],
                  taps=2, side=128, loop=(0, 4, 1), embed_scale=1.0, residual_mult=1.0, logit_scale=1.0),
    # ones: a head, an expert, a tap, a row the decays come from, values one wide; a whole model looped
    "ones": model(24, 31, [latent(1, 8, 2, 12, 6, 5, moe(1, 1, 24)), delta(1, 12, 1, moe(3, 1, 17)), latent(12, 1, 4, 1, 9, 7, neighbours=False)],
                  groups=2, taps=1, side=3, loop=(0, 3, 2), eps=1e-2),
    # norms of a single number are its sign: a column a latent row, a query row, a side part, a group, a state
    "signs": model(6, 31, [latent(2, 4, 2, 3, 1, 1, moe(2, 1, 5)), delta(3, 1, 2), latent(1, 1, 2, 1, 1, 1, neighbours=False)], groups=6, taps=2, side=1),
    # large heads, values wider and narrower than keys, states that no one block holds, many experts, many groups and taps
    "wide": model(264, 515, [latent(4, 200, 40, 72, 300, 130, moe(40, 8, 72), base=500.0), delta(2, 256, 33, moe(33, 1, 16)), delta(3, 150, 64),
                             latent(2, 64, 64, 256, 230, 512, moe(36, 6, 40), neighbours=False)], groups=6, taps=9, side=33),
    # many heads on a latent row, many small states
    "crowd": model(96, 128, [latent(70, 16, 8, 24, 140, 30, moe(9, 2, 48), scaling=stretch(8.0, 32, 4.0, 0.5)), delta(20, 48, 16, moe(8, 3, 20)),
                             latent(33, 8, 16, 16, 250, 64, neighbours=False), delta(9, 100, 8)], groups=4, taps=5, side=16, loop=(1, 2, 2)),
    # latent rows of more columns than 512, and than the tiles take
    "vast": model(64, 90, [latent(3, 16, 64, 12, 512, 40, moe(4, 2, 24)), latent(2, 24, 8, 24, 1016, 16, neighbours=False), latent(20, 8, 16, 8, 560, 8)], groups=2),
}


def weights(config, seed=0, coded=False):
    """bf16-representable fp32 tensors of unit-sized activations: matrices N(0, 1/columns), norm factors around 1, queries of a
    delta rule that lie along its keys more than not.

    `coded`: which experts a token takes is made to rest on no close call. As many of the first columns as a layer has
    experts at most (inside the first group of columns) hold a token's own permutation of evenly spaced levels, nothing adds
    to these columns, and an expert's logit is one of them, give or take a little of the rest of the row."""
    generator = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, shape in tensor_shapes(config).items():
        draw = torch.randn(shape, generator=generator)
        last = name.rsplit(".", 1)[-1]
        if last in ("w0", "b"):
            draw = 0.7 * draw
        elif last == "canon1":
            draw = 0.6 * draw / math.sqrt(shape[1])
        elif name == "side.embed":
            draw = draw
        elif len(shape) == 2:
            draw = draw if name == "embed" else draw / math.sqrt(shape[1])
        else:
            draw = 1.0 + 0.1 * draw
        tensors[name] = draw
    for index, item in enumerate(config["layers"]):
        if item["type"] == "general_delta":
            r, k = tensors[f"l{index}.mix.r"], tensors[f"l{index}.mix.k"]
            r.copy_((r + 2.0 * k) / math.sqrt(5.0))
    counts = {f"l{index}.": item["mlp"]["router"]["experts"] for index, item in enumerate(config["layers"]) if item["mlp"]}
    if coded and counts:
        most = max(counts.values())
        assert most <= config["width"] // config["norm"]["groups"]
        levels = torch.linspace(-2.0, 2.0, most)
        for token in range(config["vocab"]):
            tensors["embed"][token, :most] = levels[torch.randperm(most, generator=generator)]
        for name, tensor in tensors.items():
            if name.endswith((".mix.o", ".down", ".side.norm")):
                tensor[:most] = 0.0
            if name.endswith(".norm1"):
                tensor[:most] = 1.0
        for prefix, count in counts.items():
            router = tensors[prefix + "mlp.router"]
            router *= 0.01
            router[:, :most] = 0.0
            router[torch.arange(count), torch.randperm(most, generator=generator)[:count]] = 2.0
    return {name: tensor.to(torch.bfloat16).float() for name, tensor in tensors.items()}


def weights_for(config, dtype, seed=0):
    """In 32 bits any router will do; in bf16 the choice of experts must not hang on rounding."""
    return weights(config, seed, coded=dtype == "bf16")


def truth(config, tensors, ids):
    """(logits, residual stream per layer run) in float64, as fp32."""
    logits, kept = benarax_oracle.forward(config, tensors, ids, torch.float64)
    return logits.float(), kept.float()


TOLERANCE = {"f32": 3e-5, "bf16": 0.06}
# (which side of zero a number lies on may hang on 16-bit rounding)
RUNS = [(name, dtype) for name in sorted(CASES) for dtype in ("f32", "bf16") if name != "signs" or dtype == "f32"]
