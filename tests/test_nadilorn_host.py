"""Nadilorn on ragged-step plans without a GPU: the layer program of its config, the plan's buffer table and packing
recipes, programs that are refused, and the plain forward's mechanisms against their definitions written out."""
import json
import math
import shutil

import pytest
import torch

import nadilorn_case as case
from oracle import nadilorn_oracle as oracle
from tilemega_b200.planbuild import emit_plan
from tilemega_b200.registry import family_of, tensor_shapes
from tilemega_b200.serving.plan import RAGGED, PlanLibrary
from tilemega_b200.serving.state import allocate_ragged_state, rotary_pairs
from tilemega_b200.serving.weights import TensorCheckpoint, load_weights


def test_layer_program_takes_every_size_and_constant_from_the_config():
    config = case.CASES["odd"]
    assert family_of(config).plans == ("ragged",)
    program = family_of(config).layer_program(config)
    assert [program[key] for key in ("width", "vocab", "eps")] == [86, 203, 1e-3]
    first, second, third, _ = program["layers"]
    assert first["norm_at"] == "output" and first["norm1"] == "l0.norm1" and first["norm2"] == "l0.norm2"
    mixer = first["mixer"]
    assert [mixer[key] for key in ("heads", "kv_heads", "dim", "vdim", "values", "sink", "gate", "qk_norm")] == [9, 3, 20, 28, "projected", 0.0, True, True]
    assert mixer["rotary"] == {"base": 10000.0, "dims": 12, "factor": 2.5} and mixer["mask"] == {"size": 19}
    assert mixer["tensors"]["q.norm"] == "l0.mix.q.norm" and mixer["tensors"]["g"] == "l0.mix.g"
    experts = first["mlp"]
    assert [experts[key] for key in ("kind", "experts", "top", "ff")] == ["experts", 7, 3, 50]
    assert experts["tensors"]["up"][6] == "l0.mlp.e6.up" and experts["tensors"]["router"] == "l0.mlp.router"
    assert second["mlp"]["kind"] == "glu" and second["mlp"]["activation"] == "gelu_tanh" and second["mlp"]["ff"] == 70
    assert third["mlp"] is None and third["norm2"] is None
    assert [run["layer"] for run in program["runs"]] == [0, 1, 2, 3]
    shapes = tensor_shapes(config)
    assert shapes["l0.mix.g"] == (9 * 28, 86) and shapes["l0.mix.v"] == (3 * 28, 86) and shapes["l0.mix.o"] == (86, 9 * 28)
    assert shapes["l0.mix.k.norm"] == (60,) and shapes["l0.mlp.e2.down"] == (86, 50) and shapes["l0.mlp.router"] == (7, 86)
    assert "l2.norm2" not in shapes and "l1.mlp.gate" in shapes
    with pytest.raises(ValueError, match="unknown layer type"):
        family_of(config).layer_program(config | {"layers": [config["layers"][0] | {"type": "other"}]})
    with pytest.raises(ValueError, match="unknown feed-forward"):
        family_of(config).layer_program(config | {"layers": [config["layers"][0] | {"mlp": {"kind": "other"}}]})


@pytest.mark.parametrize("name", sorted(case.CASES))
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_buffer_table_and_recipes(name, dtype, plan_dir):
    config = case.CASES[name]
    library = PlanLibrary(emit_plan(config, plan_dir, phase="ragged", slots=3, capacity=64, num_blocks=9, max_rows=32, dtype=dtype))
    assert library.info.phase == RAGGED
    tensors = case.weights(config)
    loaded = load_weights(TensorCheckpoint(tensors), library, device="cpu")    # element counts are checked inside
    up = lambda count: -(-count // 8) * 8
    width = config["width"]
    for index, item in enumerate(config["layers"]):
        p, mixer = f"l{index}.", item["mixer"]
        stacked = loaded[p + "in.weight"].float().reshape(-1, up(width))
        assert torch.equal(stacked[:, :width], torch.cat([tensors[p + "mix." + part] for part in "qkvg"])) and not stacked[:, width:].any()
        assert torch.equal(loaded[p + "k.norm"], tensors[p + "mix.k.norm"]) and loaded[p + "q.norm"].dtype == torch.float32
        if item["mlp"] and item["mlp"]["kind"] == "moe":
            count, ff = item["mlp"]["router"]["experts"], item["mlp"]["expert"]["ff"]
            ups = loaded[p + "experts.up"].float().reshape(count, ff, up(width))
            downs = loaded[p + "experts.down"].float().reshape(count, width, up(ff))
            assert torch.equal(ups[count - 1][:, :width], tensors[f"{p}mlp.e{count - 1}.up"])
            assert torch.equal(downs[count // 2][:, :ff], tensors[f"{p}mlp.e{count // 2}.down"]) and not downs[..., ff:].any()
            assert torch.equal(loaded[p + "router.weight"].float().reshape(count, -1)[:, :width], tensors[p + "mlp.router"])
    state = allocate_ragged_state(library, "cpu")
    for index, item in enumerate(config["layers"]):
        mixer, whole = item["mixer"], lambda size: -(-size // 16) * 16
        assert state[f"kv_pool.k.{index}"].numel() == 9 * 16 * mixer["kv_heads"] * whole(mixer["dim"])
        assert state[f"kv_pool.v.{index}"].numel() == 9 * 16 * mixer["kv_heads"] * whole(mixer["vdim"])


def test_rotary_tables_by_base_dims_and_factor(plan_dir):
    """Layers share a table only if all three agree."""
    config = case.model(16, 20, [case.layer(1, 1, 8, 8, 4, 5, factor=f, base=b) for f, b in ((2.0, 50.0), (3.0, 50.0), (2.0, 50.0), (2.0, 60.0))])
    library = PlanLibrary(emit_plan(config, plan_dir, phase="ragged", slots=1, capacity=32, num_blocks=3, max_rows=8))
    state = allocate_ragged_state(library, "cpu")
    assert sorted(name for name in state if name.startswith("rotary")) == ["rotary.0", "rotary.1", "rotary.2"]
    angle = lambda table, p, i: math.atan2(*state[table].reshape(32, 2, 2)[p, i].flip(0).tolist())
    assert angle("rotary.0", 3, 0) == pytest.approx(3 / 2.0) and angle("rotary.1", 3, 0) == pytest.approx(3 / 3.0)
    assert angle("rotary.2", 7, 1) == pytest.approx(7 * 60.0 ** -0.5 / 2.0)
    assert torch.equal(rotary_pairs(50.0, 4, 32), rotary_pairs(50.0, 4, 32, 1.0))


@pytest.mark.parametrize("break_it, message", [
    (lambda l: l[0]["mixer"].update(vdim=300), "head sizes"),
    (lambda l: l[0]["mixer"]["rotary"].update(factor=0), "scaling factor"),
    (lambda l: l[0]["mixer"].update(bias=True), "no projection biases"),
    (lambda l: l[0]["mixer"].update(values="keys"), "as wide as keys"),
    (lambda l: l[0]["mlp"].update(top=8), "of a layer's experts"),
    (lambda l: l[0]["mlp"].update(experts=6), "one tensor per expert"),
    (lambda l: l[0]["mlp"].update(activation="relu"), "square of relu"),
    (lambda l: l[0]["mlp"].update(weighted="output"), "weights on their inputs"),
    (lambda l: l[1]["mlp"].update(activation="relu"), "unknown activation"),
    (lambda l: l[1].update(norm_at="input"), "same place"),
    (lambda l: l[1].update(norm_at="both"), "input or output"),
])
def test_unsupported_programs_are_refused(break_it, message, plan_dir, capfd):
    so = emit_plan(case.CASES["odd"], plan_dir, phase="ragged", slots=2, capacity=32, num_blocks=5, max_rows=16)
    document = json.loads((so.parent / (so.name + ".plan.json")).read_text())
    break_it(document["model"]["layers"])
    broken = so.parent / f"tilemega_b200_refused_{abs(hash(message)) % 10 ** 8}.so"
    shutil.copyfile(so, broken)
    (so.parent / (broken.name + ".plan.json")).write_text(json.dumps(document))
    with pytest.raises(RuntimeError, match=message):
        PlanLibrary(broken)


def test_coded_routers_rest_on_no_close_call():
    for name in ("odd", "wide", "grouped"):
        config = case.CASES[name]
        tensors, ids = case.weights(config, coded=True), case.tokens(config, 60)
        _, kept = case.truth(config, tensors, ids)
        for index, item in enumerate(config["layers"]):
            if not item["mlp"] or item["mlp"]["kind"] != "moe":
                continue
            # (what the router reads, before its own output is added, is the same in the coded columns)
            z = (kept[index] @ tensors[f"l{index}.mlp.router"].T).sort(-1, descending=True).values
            top = item["mlp"]["router"]["top"]
            assert top == z.shape[1] or (z[:, top - 1] - z[:, top]).min() > 0.004      # (rounding moves it by a few 1e-4)


# ---- the plain forward's mechanisms --------------------------------------------------------------------------------------
def draws(*shapes):
    generator = torch.Generator().manual_seed(6)
    return [torch.randn(*shape, generator=generator, dtype=torch.float64) for shape in shapes]


def test_plain_attention_is_the_sum_written_out():
    q, k, v = draws((11, 4, 6), (11, 2, 6), (11, 2, 5))
    for scale, size in ((0.4, 3), (2.0, 1), (0.1, None)):
        got = oracle.attention(q, k, v, scale, size)
        for i in range(11):
            for head in range(4):
                sees = [j for j in range(11) if j <= i and (size is None or j > i - size)]
                e = [math.exp(scale * float(q[i, head] @ k[j, head // 2])) for j in sees]
                want = sum(weight * v[j, head // 2] for weight, j in zip(e, sees)) / (1.0 + sum(e))
                assert torch.allclose(got[i, head], want)


def test_plain_softmax_with_null_is_a_softmax_with_one_more_key():
    (score,) = draws((7, 9))
    seen = score > -1.0
    seen[3] = False                                              # nothing but the null key
    for size in (1.0, 300.0):                                    # (scores far beyond what exp holds, too)
        got = oracle.softmax_with_null(score * size, seen)
        more = torch.cat((torch.zeros(7, 1, dtype=score.dtype), (score * size).masked_fill(~seen, -math.inf)), dim=1)
        assert torch.allclose(got, torch.softmax(more, dim=1)[:, 1:])
    assert not got[3].any()


def test_plain_rotation_turns_by_scaled_angles():
    (q,) = draws((1, 1, 10))
    turned = oracle.rotate(q, torch.tensor([9]), 50.0, 6, 3.0)
    for i in range(3):
        a = 9 * 50.0 ** (-2 * i / 6) / 3.0
        u, v = float(q[0, 0, i]), float(q[0, 0, i + 3])
        assert float(turned[0, 0, i]) == pytest.approx(u * math.cos(a) - v * math.sin(a))
        assert float(turned[0, 0, i + 3]) == pytest.approx(v * math.cos(a) + u * math.sin(a))
    assert torch.equal(turned[..., 6:], q[..., 6:])
    assert torch.allclose(turned, oracle.rotate(q, torch.tensor([3]), 50.0, 6))      # a third of the angle


def test_plain_window_definition():
    seen = lambda i, size: [j for j in range(i + 2) if oracle.visible(i, j, size)]
    assert seen(9, 3) == [7, 8, 9] and seen(2, 3) == [0, 1, 2] and seen(4, 1) == [4] and seen(3, None) == [0, 1, 2, 3]


def test_plain_experts():
    x, router, *matrices = draws((5, 8), (3, 8), (4, 8), (8, 4), (4, 8), (8, 4), (4, 8), (8, 4))
    named = {f"e{i // 2}.{'up' if i % 2 == 0 else 'down'}": matrix for i, matrix in enumerate(matrices)} | {"router": router}
    got = oracle.expert_mixture(x, {"router": {"top": 2}}, named.__getitem__)
    for t in range(5):
        scores = [1 / (1 + math.exp(-float(router[e] @ x[t]))) for e in range(3)]
        want = torch.zeros(8, dtype=x.dtype)
        for e in sorted(range(3), key=lambda e: -scores[e])[:2]:
            hidden = named[f"e{e}.up"] @ (scores[e] * x[t])
            want += named[f"e{e}.down"] @ torch.where(hidden > 0, hidden * hidden, torch.zeros_like(hidden))
        assert torch.allclose(got[t], want)


def test_plain_gelu_and_norm():
    (z,) = draws((50,))
    assert torch.allclose(oracle.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    x, w = draws((4, 6), (6,))
    got = oracle.rms_norm(x, w, 0.5)
    assert torch.allclose(got[2], x[2] / math.sqrt(float((x[2] ** 2).mean()) + 0.5) * w)
