"""Model families the framework serves, chosen by a model's config.json.

A family says how its models run (which kinds of plan `planbuild.emit_plan` writes for them) and, for the families
that run as ragged-step plans, how config.json becomes the layer program of such a plan's sidecar: one generic
description (mixers and feed-forwards with their constants and tensor names, and the order the layers run in) that
csrc/ragged_spec.cpp reads. A new design of known mechanisms is one more function here.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass
from pathlib import Path
from typing import Callable


@dataclass(frozen=True)
class Family:
    name: str
    plans: tuple[str, ...]                          # phases emit_plan writes for it
    layer_program: Callable[[dict], dict] | None = None
    complete: Callable[[dict, Callable], dict] | None = None   # fills in sizes only the checkpoint's tensor shapes tell


def looped_runs(count: int, loop: dict | None, add_embedding: bool = True) -> list[dict]:
    """The order `count` layers run in when layers start .. stop-1 run `times` times in a row; with `add_embedding` every
    pass but the first begins by adding the embedding output to the residual stream."""
    if not loop:
        return [{"layer": layer, "add_embedding": False} for layer in range(count)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= start <= stop <= count or times < 1:
        raise ValueError(f"loop {loop} does not fit {count} layers")
    body = [(layer, add_embedding and turn > 0 and layer == start) for turn in range(times) for layer in range(start, stop)]
    order = [(layer, False) for layer in range(start)] + body + [(layer, False) for layer in range(stop, count)]
    return [{"layer": layer, "add_embedding": again} for layer, again in order]


def _names(prefix: str, *parts: str) -> dict:
    return {part: prefix + part for part in parts}


def _bamudra_mixer(kind: str, mixer: dict, prefix: str) -> dict:
    shared = {"kind": kind, "heads": mixer["heads"], "dim": mixer["dim"], "vdim": mixer["vdim"], "rotary": mixer.get("rot")}
    if kind == "retention":
        return shared | {"decay": list(mixer["decay"]), "tensors": _names(prefix, "q", "k", "v", "g", "o")}
    if kind == "attention":
        # the values are the keys before their rotation; q, k and the output projection have biases
        return shared | {"kv_heads": mixer["kv_heads"], "values": "keys", "bias": True, "mask": mixer.get("mask"), "scale": mixer["scale"],
                         "tensors": _names(prefix, "q", "k", "o", "q.b", "k.b", "o.b")}
    raise ValueError(f"unknown layer type {kind!r}")


def _bamudra_mlp(mlp: dict | None, prefix: str) -> dict | None:
    if mlp is None:
        return None
    if mlp["kind"] != "dense":
        raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
    return {"kind": "glu", "ff": mlp["ff"], "limit": mlp["limit"], "alpha": 1.702, "shift": 1.0,
            "tensors": _names(prefix, "gate", "up", "down")}


def bamudra_program(config: dict) -> dict:
    layers = []
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{index}."
        mlp = _bamudra_mlp(layer.get("mlp"), prefix + "mlp.")
        layers.append({"norm1": prefix + "norm1", "mixer": _bamudra_mixer(layer["type"], layer["mixer"], prefix + "mix."),
                       "norm2": prefix + "norm2" if mlp else None, "mlp": mlp})
    return {"width": config["width"], "vocab": config["vocab"], "eps": config["norm"]["eps"], "embed": "embed", "final_norm": "final.norm",
            "head": "head", "layers": layers, "runs": looped_runs(len(layers), config.get("loop"))}


def _nadilorn_mixer(kind: str, mixer: dict, prefix: str) -> dict:
    if kind != "attention":
        raise ValueError(f"unknown layer type {kind!r}")
    rot = mixer.get("rot")
    rotary = rot and {"base": rot["base"], "dims": rot["dims"], "factor": (rot.get("scaling") or {}).get("factor", 1.0)}
    # queries and keys are normed before their rotation, the softmax has a null key of score 0, the heads' outputs a gate
    return {"kind": kind, "heads": mixer["heads"], "kv_heads": mixer["kv_heads"], "dim": mixer["dim"], "vdim": mixer["vdim"],
            "rotary": rotary, "mask": mixer.get("mask"), "scale": mixer["scale"], "values": "projected", "qk_norm": True, "sink": 0.0,
            "gate": True, "tensors": _names(prefix, "q", "k", "v", "g", "o", "q.norm", "k.norm")}


def _nadilorn_mlp(mlp: dict | None, prefix: str) -> dict | None:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return {"kind": "glu", "ff": mlp["ff"], "activation": "gelu_tanh", "tensors": _names(prefix, "gate", "up", "down")}
    if mlp["kind"] != "moe":
        raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
    count = int(mlp["router"]["experts"])
    # a token's scores weigh the rows its experts read, as they are
    return {"kind": "experts", "ff": mlp["expert"]["ff"], "experts": count, "top": mlp["router"]["top"], "activation": "relu2",
            "scores": "sigmoid", "weighted": "input",
            "tensors": {"router": prefix + "router"} | {part: [f"{prefix}e{expert}.{part}" for expert in range(count)] for part in ("up", "down")}}


def nadilorn_program(config: dict) -> dict:
    layers = []
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{index}."
        mlp = _nadilorn_mlp(layer.get("mlp"), prefix + "mlp.")
        layers.append({"norm_at": "output", "norm1": prefix + "norm1", "mixer": _nadilorn_mixer(layer["type"], layer["mixer"], prefix + "mix."),
                       "norm2": prefix + "norm2" if mlp else None, "mlp": mlp})
    return {"width": config["width"], "vocab": config["vocab"], "eps": config["norm"]["eps"], "embed": "embed", "final_norm": "final.norm",
            "head": "head", "layers": layers, "runs": looped_runs(len(layers), None)}


def _mozidra_mixer(kind: str, mixer: dict, prefix: str, first_mixing: bool) -> dict:
    shared = {"heads": mixer["heads"], "dim": mixer["dim"], "vdim": mixer["vdim"], "mask": mixer.get("mask"), "scale": mixer["scale"]}
    if kind == "latent_attention":
        return shared | {"kind": "latent", "rank": mixer["kv_rank"], "tensors": _names(prefix, "q", "dkv", "dkv.norm", "uk", "uv", "sink", "o")}
    if kind != "attention":
        raise ValueError(f"unknown layer type {kind!r}")
    # biased projections, normed queries and keys, rotated pairs of neighbours, a learned sink per head; layers that mix
    # values blend their own with those of the first such layer
    rot, mixing = mixer.get("rot"), mixer.get("v_mix")
    tensors = _names(prefix, "q", "k", "v", "o", "q.b", "k.b", "v.b", "q.norm", "k.norm", "sink")
    if mixing and not first_mixing:
        tensors |= _names(prefix, "vmix")
    return shared | {"kind": kind, "kv_heads": mixer["kv_heads"], "rotary": rot and {"base": rot["base"], "dims": rot["dims"], "layout": "pairs"},
                     "values": "projected", "qk_norm": True, "bias": True, "value_mix": ("source" if first_mixing else "blend") if mixing else "",
                     "tensors": tensors}


def _mozidra_mlp(mlp: dict | None, prefix: str) -> dict | None:
    if mlp is None:
        return None
    if mlp["kind"] != "moe":
        raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
    router, shared = mlp["router"], mlp.get("shared")
    count = int(router["experts"])
    tensors = _names(prefix, "router", "correction") | {part: [f"{prefix}e{expert}.{part}" for expert in range(count)] for part in ("gate", "up", "down")}
    if shared:
        tensors |= _names(prefix, "shared.gate", "shared.up", "shared.down", "shared.sg")
    return {"kind": "experts", "ff": mlp["expert"]["ff"], "limit": mlp["expert"]["limit"], "alpha": 1.702, "shift": 1.0, "experts": count,
            "top": router["top"], "groups": router.get("groups"), "activation": "silu", "scores": "softmax", "weighted": "output",
            "shared": shared and {"ff": shared["ff"], "limit": shared["limit"]}, "tensors": tensors}


def mozidra_program(config: dict) -> dict:
    layers, mixing = [], [index for index, layer in enumerate(config["layers"]) if layer["mixer"].get("v_mix")]
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{index}."
        mlp = _mozidra_mlp(layer.get("mlp"), prefix + "mlp.")
        layers.append({"norm1": prefix + "norm1", "norm2": prefix + "norm2" if mlp else None, "mlp": mlp,
                       "mixer": _mozidra_mixer(layer["type"], layer["mixer"], prefix + "mix.", index in mixing[:1]),
                       "streams": [_names(f"{prefix}hc{number}.", "in", "out", "mix") for number in ((1, 2) if mlp else (1,))]})
    # stored norm weights are distances from one
    return {"width": config["width"], "vocab": config["vocab"], "eps": config["norm"]["eps"], "norm_offset": 1.0, "streams": config["streams"],
            "embed": "embed", "final_norm": "final.norm", "head": "head", "layers": layers, "runs": looped_runs(len(layers), None)}


def _benarax_mixer(kind: str, mixer: dict, prefix: str) -> dict:
    if kind == "general_delta":
        # decay_rank: a completed config has it, see complete_benarax
        return {"kind": "delta", "heads": mixer["heads"], "dim": mixer["dim"], "decay_rank": mixer["decay_rank"], "decay_scale": math.exp(-0.5),
                "unit_eps": 1e-6, "tensors": _names(prefix, "r", "k", "v", "a", "a.b", "g", "w1", "w2", "w0", "norm", "o")}
    if kind not in ("latent_attention", "latent_attention_2"):
        raise ValueError(f"unknown layer type {kind!r}")
    rot = mixer["rot"]
    if rot["dims"] != mixer["rot_dim"]:
        raise ValueError("the whole rotated part of a head turns")
    # the two kinds differ in which entries of the rotated part turn together
    return {"kind": "latent", "heads": mixer["heads"], "dim": mixer["dim"], "vdim": mixer["vdim"], "rank": mixer["kv_rank"], "q_rank": mixer["q_rank"],
            "rotary": {"base": rot["base"], "dims": rot["dims"], "layout": "pairs" if kind == "latent_attention" else "halves", "yarn": rot.get("scaling")},
            "scale": mixer["scale"], "tensors": _names(prefix, "dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "o")}


def _benarax_mlp(mlp: dict | None, prefix: str) -> dict | None:
    if mlp is None:
        return None
    if mlp["kind"] != "moe":
        raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
    count = int(mlp["router"]["experts"])
    return {"kind": "experts", "ff": mlp["expert"]["ff"], "limit": mlp["expert"]["limit"], "alpha": 1.702, "shift": 1.0, "experts": count,
            "top": mlp["router"]["top"], "activation": "silu", "scores": "softmax_chosen", "weighted": "output",
            "tensors": {"router": prefix + "router"} | {part: [f"{prefix}e{expert}.{part}" for expert in range(count)] for part in ("gate", "up", "down")}}


def benarax_program(config: dict) -> dict:
    layers, side = [], config["token_side"]
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{index}."
        layers.append({"norm1": prefix + "norm1", "mixer": _benarax_mixer(layer["type"], layer["mixer"], prefix + "mix."),
                       "mlp": _benarax_mlp(layer.get("mlp"), prefix + "mlp."), "conv": prefix + "canon1",
                       "side": _names(prefix + "side.", "gate", "proj", "norm") | {"from": index * side["dim"]}})
    return {"width": config["width"], "vocab": config["vocab"], "eps": config["norm"]["eps"], "form": "parallel", "norm_groups": config["norm"]["groups"],
            "taps": config["canon"]["taps"], "residual_mult": config["residual_mult"], "embed_scale": config["embedding"]["scale"],
            "logit_scale": config["logit_scale"], "side": {"embed": "side.embed", "dim": side["dim"]}, "embed": "embed", "final_norm": "final.norm",
            "head": "head", "layers": layers, "runs": looped_runs(len(layers), config.get("loop"), add_embedding=False)}


def complete_benarax(config: dict, shape_of: Callable) -> dict:
    """The decays of a delta rule come through a row whose size no key of the config gives: that of the tensor."""
    layers = []
    for index, layer in enumerate(config["layers"]):
        if layer["type"] == "general_delta" and "decay_rank" not in layer["mixer"]:
            layer = layer | {"mixer": layer["mixer"] | {"decay_rank": int(shape_of(f"l{index}.mix.w1")[0])}}
        layers.append(layer)
    return config | {"layers": layers}


FAMILIES = {
    "LlamaForCausalLM": Family("llama", ("decode", "prefill")),
    "Qwen3MoeForCausalLM": Family("qwen3-moe", ("decode",)),
    "BertModel": Family("bert", ("forward",)),
    "Bamudra": Family("bamudra", ("ragged",), bamudra_program),
    "Nadilorn": Family("nadilorn", ("ragged",), nadilorn_program),
    "Mozidra": Family("mozidra", ("ragged",), mozidra_program),
    "Benarax": Family("benarax", ("ragged",), benarax_program, complete_benarax),
}


def architecture_of(config: dict) -> str:
    if "architecture" in config:
        return str(config["architecture"])
    names = config.get("architectures") or ["LlamaForCausalLM"]
    return str(names[0])


def family_of(config: dict) -> Family:
    name = architecture_of(config)
    if name not in FAMILIES:
        raise ValueError(f"no model family serves {name!r} (known: {', '.join(sorted(FAMILIES))})")
    return FAMILIES[name]


def load_config(model_dir: str | Path) -> dict:
    """config.json of a model folder, with the sizes its family takes from the checkpoint's tensor shapes."""
    config = json.loads((Path(model_dir) / "config.json").read_text())
    complete = FAMILIES[architecture_of(config)].complete if architecture_of(config) in FAMILIES else None
    if complete is None:
        return config
    from .serving.weights import Checkpoint
    return complete(config, Checkpoint(model_dir).shape)


def vocab_of(config: dict) -> int:
    return int(config["vocab"] if "vocab" in config else config["vocab_size"])


def tensor_shapes(config: dict) -> dict[str, tuple[int, ...]]:
    """Checkpoint tensors (name -> shape) a layer program reads."""
    program = family_of(config).layer_program(config)
    width, shapes = program["width"], {}
    shapes[program["embed"]] = (program["vocab"], width)
    for layer in program["layers"]:
        mixer, names = layer["mixer"], layer["mixer"]["tensors"]
        heads, streams = mixer["heads"], program.get("streams", 1)
        vdim = mixer.get("vdim", mixer["dim"])
        q, out = heads * mixer["dim"], heads * vdim
        k, rank, turned = mixer.get("kv_heads", heads) * mixer["dim"], mixer.get("rank", 0), (mixer.get("rotary") or {}).get("dims", 0)
        q_rank, decay_rank = mixer.get("q_rank", 0), mixer.get("decay_rank", 0)
        sizes = {"q": q, "k": k, "v": mixer.get("kv_heads", heads) * vdim, "g": out, "dkv": rank + (turned if q_rank else 0), "dq": q_rank, "r": q,
                 "a": q, "w1": decay_rank, "o": width}
        special = {"o": (width, out), "uk": (q, rank), "uv": (out, rank), "uq": (q + heads * turned, q_rank), "sink": (heads,), "vmix": (),
                   "dkv.norm": (rank,), "w2": (q, decay_rank), "w0": (q,), "norm": (out,)}
        shapes[layer["norm1"]] = (width,)
        for part, name in names.items():
            if part in special:
                shapes[name] = special[part]
            elif part.endswith((".norm", ".b")):
                shapes[name] = (sizes[part.rsplit(".", 1)[0]],)
            else:
                shapes[name] = (sizes[part], width)
        if program.get("taps"):
            shapes[layer["conv"]] = (width, program["taps"])
        if "side" in layer:
            part = program["side"]["dim"]
            shapes |= {layer["side"]["gate"]: (part, width), layer["side"]["proj"]: (width, part), layer["side"]["norm"]: (width,)}
        for parts in layer.get("streams", ()):
            shapes |= {parts["in"]: (streams,), parts["out"]: (streams,), parts["mix"]: (streams, streams)}
        if layer["mlp"]:
            ff, parts = layer["mlp"]["ff"], layer["mlp"]["tensors"]
            if "norm2" in layer:
                shapes[layer["norm2"]] = (width,)
            if layer["mlp"]["kind"] == "experts":
                shapes[parts["router"]] = (layer["mlp"]["experts"], width)
                shapes |= {name: (ff, width) for part in ("gate", "up") for name in parts.get(part, ())} | {name: (width, ff) for name in parts["down"]}
                if "correction" in parts:
                    shapes[parts["correction"]] = (layer["mlp"]["experts"],)
                if layer["mlp"].get("shared"):
                    wide = layer["mlp"]["shared"]["ff"]
                    shapes |= {parts["shared.gate"]: (wide, width), parts["shared.up"]: (wide, width), parts["shared.down"]: (width, wide),
                               parts["shared.sg"]: (1, width)}
            else:
                shapes |= {parts["gate"]: (ff, width), parts["up"]: (ff, width), parts["down"]: (width, ff)}
    if "side" in program:
        shapes[program["side"]["embed"]] = (program["vocab"], program["side"]["dim"] * len(program["layers"]))
    shapes[program["final_norm"]] = (width,)
    shapes[program["head"]] = (program["vocab"], width)
    return shapes
