"""Model families the framework serves, chosen by a model's config.json.

A family says how its models run (which kinds of plan `planbuild.emit_plan` writes for them) and, for the families
that run as ragged-step plans, how config.json becomes the layer program of such a plan's sidecar: one generic
description (mixers and feed-forwards with their constants and tensor names, and the order the layers run in) that
csrc/ragged_spec.cpp reads. A new design of known mechanisms is one more function here.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable


@dataclass(frozen=True)
class Family:
    name: str
    plans: tuple[str, ...]                          # phases emit_plan writes for it
    layer_program: Callable[[dict], dict] | None = None


def looped_runs(count: int, loop: dict | None) -> list[dict]:
    """The order `count` layers run in when layers start .. stop-1 run `times` times in a row; every pass but the
    first begins by adding the embedding output to the residual stream."""
    if not loop:
        return [{"layer": layer, "add_embedding": False} for layer in range(count)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= start <= stop <= count or times < 1:
        raise ValueError(f"loop {loop} does not fit {count} layers")
    body = [(layer, turn > 0 and layer == start) for turn in range(times) for layer in range(start, stop)]
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


FAMILIES = {
    "LlamaForCausalLM": Family("llama", ("decode", "prefill")),
    "Qwen3MoeForCausalLM": Family("qwen3-moe", ("decode",)),
    "BertModel": Family("bert", ("forward",)),
    "Bamudra": Family("bamudra", ("ragged",), bamudra_program),
    "Nadilorn": Family("nadilorn", ("ragged",), nadilorn_program),
    "Mozidra": Family("mozidra", ("ragged",), mozidra_program),
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
    return json.loads((Path(model_dir) / "config.json").read_text())


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
        q, out = heads * mixer["dim"], heads * mixer["vdim"]
        k, rank = mixer.get("kv_heads", heads) * mixer["dim"], mixer.get("rank", 0)
        sizes = {"q": q, "k": k, "v": mixer.get("kv_heads", heads) * mixer["vdim"], "g": out, "dkv": rank, "o": width}
        special = {"o": (width, out), "uk": (q, rank), "uv": (out, rank), "sink": (heads,), "vmix": ()}
        shapes[layer["norm1"]] = (width,)
        for part, name in names.items():
            if part.endswith((".norm", ".b")):
                shapes[name] = (sizes[part.rsplit(".", 1)[0]],)
            else:
                shapes[name] = special[part] if part in special else (sizes[part], width)
        for parts in layer.get("streams", ()):
            shapes |= {parts["in"]: (streams,), parts["out"]: (streams,), parts["mix"]: (streams, streams)}
        if layer["mlp"]:
            ff, parts = layer["mlp"]["ff"], layer["mlp"]["tensors"]
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
    shapes[program["final_norm"]] = (width,)
    shapes[program["head"]] = (program["vocab"], width)
    return shapes
