"""Mozidra on ragged-step plans without a GPU: the layer program of its config, the plan's buffer table and packing
recipes, programs that are refused, and the plain forward's mechanisms against their definitions written out."""
import json
import math
import shutil

import pytest
import torch

import mozidra_case as case
from oracle import mozidra_oracle as oracle
from tilemega_b200.planbuild import emit_plan
from tilemega_b200.registry import family_of, tensor_shapes
from tilemega_b200.serving.plan import RAGGED, PlanLibrary
from tilemega_b200.serving.state import allocate_ragged_state
from tilemega_b200.serving.weights import TensorCheckpoint, load_weights, per_head


def test_layer_program_takes_every_size_and_constant_from_the_config():
    config = case.CASES["odd"]
    assert family_of(config).plans == ("ragged",)
    program = family_of(config).layer_program(config)
    assert [program[key] for key in ("width", "vocab", "eps", "streams", "norm_offset")] == [86, 203, 1e-3, 3, 1.0]
    first, second, third, fourth, fifth, _ = program["layers"]
    assert [first["mixer"][key] for key in ("kind", "heads", "dim", "vdim", "rank", "mask")] == ["latent", 5, 20, 28, 43, {"size": 19}]
    assert first["mixer"]["tensors"]["dkv.norm"] == "l0.mix.dkv.norm" and "rotary" not in first["mixer"]
    assert first["streams"] == [{part: f"l0.hc{number}.{part}" for part in ("in", "out", "mix")} for number in (1, 2)]
    mixer = second["mixer"]
    assert [mixer[key] for key in ("kind", "heads", "kv_heads", "dim", "vdim", "qk_norm", "bias")] == ["attention", 9, 3, 20, 28, True, True]
    assert mixer["rotary"] == {"base": 10000.0, "dims": 12, "layout": "pairs"}
    # the first layer that mixes values is what the others blend in; one that does not say so does neither
    assert [layer["mixer"].get("value_mix") for layer in program["layers"]] == [None, "source", "", None, "blend", None]
    assert "vmix" not in mixer["tensors"] and fifth["mixer"]["tensors"]["vmix"] == "l4.mix.vmix"
    experts = first["mlp"]
    assert [experts[key] for key in ("experts", "top", "ff", "limit", "groups")] == [9, 3, 50, 1.5, {"count": 3, "keep": 2}]
    assert experts["shared"] == {"ff": 70, "limit": 0.8} and experts["tensors"]["gate"][8] == "l0.mlp.e8.gate"
    assert third["mlp"] is None and third["norm2"] is None and len(third["streams"]) == 1
    shapes = tensor_shapes(config)
    assert shapes["l0.mix.uk"] == (100, 43) and shapes["l0.mix.uv"] == (140, 43) and shapes["l0.mix.dkv"] == (43, 86) and shapes["l0.mix.sink"] == (5,)
    assert shapes["l1.mix.v.b"] == (84,) and shapes["l4.mix.vmix"] == () and "l1.mix.vmix" not in shapes and shapes["l1.mix.o"] == (86, 9 * 28)
    assert shapes["l0.hc2.mix"] == (3, 3) and "l2.hc2.mix" not in shapes and shapes["l0.mlp.shared.sg"] == (1, 86) and shapes["l0.mlp.correction"] == (9,)
    with pytest.raises(ValueError, match="unknown layer type"):
        family_of(config).layer_program(config | {"layers": [config["layers"][0] | {"type": "other"}]})
    with pytest.raises(ValueError, match="unknown feed-forward"):
        family_of(config).layer_program(config | {"layers": [config["layers"][0] | {"mlp": {"kind": "dense"}}]})


@pytest.mark.parametrize("name", sorted(case.CASES))
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_buffer_table_and_recipes(name, dtype, plan_dir):
    config = case.CASES[name]
    library = PlanLibrary(emit_plan(config, plan_dir, phase="ragged", slots=3, capacity=64, num_blocks=9, max_rows=32, dtype=dtype))
    assert library.info.phase == RAGGED
    tensors = case.weights(config)
    loaded = load_weights(TensorCheckpoint(tensors), library, device="cpu")    # element counts are checked inside
    up = lambda count, unit=8: -(-count // unit) * unit
    width = config["width"]
    assert torch.equal(loaded["final.norm"], 1.0 + tensors["final.norm"])
    for index, item in enumerate(config["layers"]):
        p, mixer = f"l{index}.", item["mixer"]
        heads, dim, vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
        assert torch.equal(loaded[p + "norm1"], 1.0 + tensors[p + "norm1"]) and torch.equal(loaded[p + "sinks"], tensors[p + "mix.sink"])
        assert torch.equal(loaded[p + "streams1.mix"], tensors[p + "hc1.mix"])
        stacked = loaded[p + "in.weight"].float().reshape(-1, up(width))
        assert not stacked[:, width:].any()
        if item["type"] == "latent_attention":
            rank, step = mixer["kv_rank"], up(dim)
            assert torch.equal(stacked[heads * step:, :width], tensors[p + "mix.dkv"])
            assert torch.equal(stacked[:heads * step, :width].reshape(heads, step, width)[:, :dim].reshape(-1, width), tensors[p + "mix.q"])
            # a query against latent rows: the head's key matrix transposed
            turned = loaded[p + "key_up.weight"].float().reshape(heads, up(rank), step)
            assert torch.equal(turned[heads - 1, :rank, :dim], tensors[p + "mix.uk"].reshape(heads, dim, rank)[heads - 1].T)
            assert not turned[:, rank:].any() and not turned[:, :, dim:].any()
            values = loaded[p + "value_up.weight"].float().reshape(heads * vdim, up(rank))
            assert torch.equal(values[:, :rank], tensors[p + "mix.uv"]) and not values[:, rank:].any()
            if dtype == "bf16":
                expanded = loaded[p + "expand.weight"].float().reshape(-1, up(rank))
                keys, rest = expanded[:heads * up(dim, 16)].reshape(heads, -1, up(rank)), expanded[heads * up(dim, 16):].reshape(heads, -1, up(rank))
                assert torch.equal(keys[:, :dim, :rank].reshape(-1, rank), tensors[p + "mix.uk"]) and not keys[:, dim:].any()
                assert torch.equal(rest[:, :vdim, :rank].reshape(-1, rank), tensors[p + "mix.uv"]) and not rest[:, vdim:].any()
        else:
            # neighbours that turn together lie half a rotation apart, in weights, biases and norms alike
            rot, q = mixer["rot"]["dims"], stacked[:heads * dim, :width].reshape(heads, dim, width)
            original = tensors[p + "mix.q"].reshape(heads, dim, width)
            assert torch.equal(q[:, 1], original[:, 2 if rot > 2 else 1]) and torch.equal(q[:, rot // 2], original[:, 1]) and torch.equal(q[:, rot:], original[:, rot:])
            bias = loaded[p + "in.bias"][:heads * dim].reshape(heads, dim)
            norm = loaded[p + "q.norm"].reshape(heads, dim)
            assert torch.equal(bias[:, rot // 2], tensors[p + "mix.q.b"].reshape(heads, dim)[:, 1])
            assert torch.equal(norm[:, rot // 2], tensors[p + "mix.q.norm"].reshape(heads, dim)[:, 1])
            assert torch.equal(stacked[(heads + mixer["kv_heads"]) * dim:, :width], tensors[p + "mix.v"])
        if item["mlp"]:
            count, ff, shared = item["mlp"]["router"]["experts"], item["mlp"]["expert"]["ff"], item["mlp"]["shared"]["ff"]
            units = loaded[p + "experts.gate_up"].float().reshape(count, -1, 2, 16, up(width))
            last = units[count - 1][:, 1].reshape(-1, up(width))[:ff, :width]
            assert torch.equal(last, tensors[f"{p}mlp.e{count - 1}.up"])
            assert torch.equal(units[0][:, 0].reshape(-1, up(width))[:ff, :width], tensors[p + "mlp.e0.gate"])
            router = loaded[p + "router.weight"].float().reshape(count + 1, -1)[:, :width]
            assert torch.equal(router[:count], tensors[p + "mlp.router"]) and torch.equal(router[count:], tensors[p + "mlp.shared.sg"])
            down = loaded[p + "shared.down"].float().reshape(width, up(shared))
            assert torch.equal(down[:, :shared], tensors[p + "mlp.shared.down"]) and torch.equal(loaded[p + "correction"], tensors[p + "mlp.correction"])
    state = allocate_ragged_state(library, "cpu")
    for index, item in enumerate(config["layers"]):
        mixer, whole = item["mixer"], lambda size: up(size, 16)
        if item["type"] == "latent_attention":
            assert state[f"kv_pool.latent.{index}"].numel() == 9 * 16 * whole(mixer["kv_rank"]) and f"kv_pool.k.{index}" not in state
        else:
            assert state[f"kv_pool.k.{index}"].numel() == 9 * 16 * mixer["kv_heads"] * whole(mixer["dim"])


@pytest.mark.parametrize("break_it, message", [
    (lambda l: l[0]["mixer"].update(vdim=300), "head sizes"),
    (lambda l: l[0]["mixer"].update(rank=1025), "1..1024 columns"),
    (lambda l: l[0]["mixer"].update(bias=True), "per head and no biases"),
    (lambda l: l[0]["mixer"].update(mask={"size": 5, "keep_first": 2}), "keeps no first positions"),
    (lambda l: l[1]["mixer"].update(values="keys", vdim=20), "halves turn"),
    (lambda l: l[1]["mixer"].update(value_mix="other"), "way of mixing"),
    (lambda l: l[1]["mixer"].update(value_mix=""), "one layer before"),
    (lambda l: l[2]["mixer"].update(value_mix="source"), "one layer before|as many of them"),
    (lambda l: l[4]["mixer"].update(vdim=15), "as many of them"),
    (lambda l: l[0]["mlp"].update(groups={"count": 2, "keep": 1}), "equal groups"),
    (lambda l: l[0]["mlp"].update(groups={"count": 9, "keep": 2}), "hold the experts of a token"),
    (lambda l: l[0]["mlp"].update(scores="other"), "softmax or sigmoid"),
    (lambda l: l[0]["mlp"].update(experts=6), "one tensor per expert|equal groups"),
    (lambda l: l[0].update(streams=[]), "each of its sublayers"),
    (lambda l: l[3].pop("streams"), "how its sublayers use them"),
    (lambda l: l[0].update(norm_at="output"), "norms on their outputs have one stream"),
])
def test_unsupported_programs_are_refused(break_it, message, plan_dir, capfd):
    so = emit_plan(case.CASES["odd"], plan_dir, phase="ragged", slots=2, capacity=32, num_blocks=5, max_rows=16)
    document = json.loads((so.parent / (so.name + ".plan.json")).read_text())
    break_it(document["model"]["layers"])
    broken = so.parent / f"tilemega_b200_refused_mozidra_{abs(hash(message)) % 10 ** 8}.so"
    shutil.copyfile(so, broken)
    (so.parent / (broken.name + ".plan.json")).write_text(json.dumps(document))
    with pytest.raises(RuntimeError, match=message):
        PlanLibrary(broken)


def test_recipes_per_head():
    matrix = torch.arange(24.0).reshape(6, 4)
    padded = per_head({"kind": "pad_heads", "heads": 2, "rows": 5}, matrix)
    assert padded.shape == (10, 4) and torch.equal(padded[5:8], matrix[3:]) and not padded[3:5].any()
    turned = per_head({"kind": "transpose_heads", "heads": 2, "rows": 3}, matrix)
    assert torch.equal(turned, torch.cat((matrix[:3].T, matrix[3:].T)))
    vector = torch.arange(10.0)
    assert per_head({"kind": "pairs_to_halves", "heads": 2, "dims": 4}, vector).tolist() == [0, 2, 1, 3, 4, 5, 7, 6, 8, 9]
    for recipe in ({"kind": "pad_heads", "heads": 4, "rows": 5}, {"kind": "pad_heads", "heads": 2, "rows": 2}, {"kind": "transpose_heads", "heads": 2, "rows": 2},
                   {"kind": "pairs_to_halves", "heads": 2, "dims": 3}):
        with pytest.raises(ValueError):
            per_head(recipe, matrix)


def test_coded_routers_rest_on_no_close_call():
    for name in ("odd", "wide", "crowd"):
        config = case.CASES[name]
        tensors, ids = case.weights(config, coded=True), case.tokens(config, 40)
        gaps = []
        original = oracle.route

        def watched(z, correction, top, groups, keep):
            score = torch.softmax(z, -1)
            rank, size = score + correction, len(z) // groups
            at = torch.stack([g * size + rank[g * size:(g + 1) * size].argmax() for g in range(groups)])
            order = at[rank[at].argsort(descending=True)]

            def gap(a, b):                       # what separates two ranks, in units of what rounding moves: the scores' size
                gaps.append(float((rank[a] - rank[b]) / torch.maximum(score[a], score[b])))

            if keep < groups:
                gap(order[keep - 1], order[keep])
            members = torch.cat([torch.arange(g * size, (g + 1) * size) for g in (order[:keep] // size).tolist()])
            members = members[rank[members].argsort(descending=True)]
            if top < len(members):
                gap(members[top - 1], members[top])
            return original(z, correction, top, groups, keep)

        oracle.route = watched
        try:
            case.truth(config, tensors, ids)
        finally:
            oracle.route = original
        assert min(gaps) > 0.02, (name, min(gaps))            # (rounding moves scores by a few 1e-3 of their size)


# ---- the plain forward's mechanisms --------------------------------------------------------------------------------------
def draws(*shapes):
    generator = torch.Generator().manual_seed(6)
    return [torch.randn(*shape, generator=generator, dtype=torch.float64) for shape in shapes]


def test_plain_attention_is_the_sum_written_out():
    q, k, v, sinks = draws((11, 4, 6), (11, 2, 6), (11, 2, 5), (4,))
    for scale, size in ((0.4, 3), (2.0, 1), (0.1, None)):
        got = oracle.attend(q, k, v, scale, size, sinks)
        for i in range(11):
            for head in range(4):
                sees = [j for j in range(11) if j <= i and (size is None or j > i - size)]
                e = [math.exp(scale * float(q[i, head] @ k[j, head // 2])) for j in sees]
                want = sum(weight * v[j, head // 2] for weight, j in zip(e, sees)) / (math.exp(float(sinks[head])) + sum(e))
                assert torch.allclose(got[i, head], want)


def test_plain_latent_mixer_against_latent_rows_themselves():
    """Expanded keys and values, and queries and sums against the latent rows, are the same attention."""
    spec = {"heads": 3, "dim": 4, "vdim": 5, "scale": 0.3, "mask": {"size": 4}}
    h, q, dkv, norm, uk, uv, sinks, o = draws((9, 10), (12, 10), (7, 10), (7,), (12, 7), (15, 7), (3,), (10, 15))
    named = {"q": q, "dkv": dkv, "dkv.norm": norm, "uk": uk, "uv": uv, "sink": sinks, "o": o}
    got = oracle.latent_mixer(h, spec, named.__getitem__, 1e-4)
    c = (h @ dkv.T) / ((h @ dkv.T).pow(2).mean(-1, keepdim=True) + 1e-4).sqrt() * norm
    lookup = torch.einsum("thd,hdr->thr", (h @ q.T).reshape(9, 3, 4), uk.reshape(3, 4, 7))
    summed = oracle.attend(lookup, c[:, None], c[:, None], 0.3, 4, sinks)
    want = torch.einsum("thr,hvr->thv", summed, uv.reshape(3, 5, 7)).reshape(9, 15) @ o.T
    assert torch.allclose(got, want)


def test_plain_rotation_turns_neighbours():
    (q,) = draws((1, 1, 10))
    turned = oracle.rotate_pairs(q, torch.tensor([9]), 50.0, 6)
    for i in range(3):
        a = 9 * 50.0 ** (-2 * i / 6)
        u, v = float(q[0, 0, 2 * i]), float(q[0, 0, 2 * i + 1])
        assert float(turned[0, 0, 2 * i]) == pytest.approx(u * math.cos(a) - v * math.sin(a))
        assert float(turned[0, 0, 2 * i + 1]) == pytest.approx(v * math.cos(a) + u * math.sin(a))
    assert torch.equal(turned[..., 6:], q[..., 6:])


def test_plain_streams():
    x, mix, out, y = draws((3, 5, 4), (3, 3), (3,), (5, 4))
    got = oracle.distribute(x, mix, out, y)
    for t in range(3):
        assert torch.allclose(got[t], mix[0, t] * x[0] + mix[1, t] * x[1] + mix[2, t] * x[2] + out[t] * y)
    assert torch.allclose(oracle.collect(x, out), out[0] * x[0] + out[1] * x[1] + out[2] * x[2])


def test_plain_values_blend_with_the_first_layers():
    spec = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 3, "scale": 0.5, "mask": {"size": 1}}
    h, first = draws((4, 6), (4, 3))
    named = {"vmix": torch.tensor(0.25, dtype=torch.float64), "sink": torch.full((2,), -50.0, dtype=torch.float64), "o": torch.eye(6, dtype=torch.float64)}
    for part, rows in (("q", 8), ("k", 4), ("v", 3)):
        named[part], named[part + ".b"], named[part + ".norm"] = *draws((rows, 6), (rows,)), torch.ones(rows, dtype=torch.float64)
    out, own = oracle.attention_mixer(h, torch.arange(4), spec, named.__getitem__, 1e-5, first)
    assert torch.allclose(own, h @ named["v"].T + named["v.b"])
    assert torch.allclose(out, (0.75 * own + 0.25 * first).repeat(1, 2))      # a window of one position: each sees its own value


def test_plain_routing():
    z = torch.log(torch.tensor([0.05, 0.30, 0.10, 0.20, 0.25, 0.10], dtype=torch.float64))
    none = torch.zeros(6, dtype=torch.float64)
    assert oracle.route(z, none, 2, 1, 1)[0] == [1, 4]
    chosen, weights = oracle.route(z, none, 2, 3, 1)                          # groups (0 1) (2 3) (4 5): only the first is open
    assert chosen == [1, 0] and [float(w) for w in weights] == pytest.approx([0.3 / 0.35, 0.05 / 0.35])
    lifted = torch.tensor([0.0, 0.0, 0.5, 0.0, 0.0, 0.0], dtype=torch.float64)
    chosen, weights = oracle.route(z, lifted, 3, 3, 2)                        # ranks are lifted, weights are not
    assert chosen == [2, 1, 3] and [float(w) for w in weights] == pytest.approx([0.1 / 0.6, 0.3 / 0.6, 0.2 / 0.6])
    sunk = torch.full((6,), -1.0, dtype=torch.float64)                        # ranks below 0 still beat closed groups
    assert oracle.route(z, sunk, 2, 3, 1)[0] == [1, 0]


def test_plain_clipped_unit():
    h, gate, up, down = draws((30, 8), (5, 8), (5, 8), (8, 5))
    got = oracle.clipped_unit(h, 0.7, {"gate": gate, "up": up, "down": down}.__getitem__)
    want = torch.zeros(5, dtype=torch.float64)
    for j in range(5):
        g, u = min(float(gate[j] @ h[3]), 0.7), max(-0.7, min(0.7, float(up[j] @ h[3])))
        want[j] = g / (1 + math.exp(-1.702 * g)) * (u + 1)
    assert torch.allclose(got[3], down @ want)
