"""Benarax on ragged-step plans without a GPU: the layer program of its config, the plan's buffer table and packing
recipes, programs that are refused, and the plain forward's mechanisms against their definitions written out."""
import json
import math
import shutil

import pytest
import torch

import benarax_case as case
from oracle import benarax_oracle as oracle
from tilemega_b200.planbuild import emit_plan
from tilemega_b200.registry import family_of, load_config, looped_runs, tensor_shapes
from tilemega_b200.serving.plan import RAGGED, PlanLibrary
from tilemega_b200.serving.state import allocate_ragged_state, rotary_pairs
from tilemega_b200.serving.weights import TensorCheckpoint, load_weights, pack, per_head


def test_layer_program_takes_every_size_and_constant_from_the_config():
    config = case.CASES["odd"]
    assert family_of(config).plans == ("ragged",)
    program = family_of(config).layer_program(config)
    assert [program[key] for key in ("width", "vocab", "eps", "form", "norm_groups", "taps")] == [90, 203, 2e-2, "parallel", 3, 4]
    assert [program[key] for key in ("residual_mult", "embed_scale", "logit_scale", "side")] == [0.8, 1.5, 0.5, {"embed": "side.embed", "dim": 7}]
    first, second, third, fourth, fifth = program["layers"]
    assert [first["mixer"][key] for key in ("kind", "heads", "dim", "vdim", "rank", "q_rank", "scale")] == ["latent", 5, 20, 28, 43, 21, 26 ** -0.5]
    assert first["mixer"]["rotary"] == {"base": 10000.0, "dims": 6, "layout": "pairs", "yarn": None}
    assert third["mixer"]["rotary"] == {"base": 300.0, "dims": 10, "layout": "halves", "yarn": None}
    assert fifth["mixer"]["rotary"]["yarn"] == {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
    assert [second["mixer"][key] for key in ("kind", "heads", "dim", "decay_rank")] == ["delta", 3, 22, 5]
    assert second["mixer"]["decay_scale"] == pytest.approx(0.6065306597) and second["mixer"]["tensors"]["a.b"] == "l1.mix.a.b"
    assert first["conv"] == "l0.canon1" and fifth["side"] == {"gate": "l4.side.gate", "proj": "l4.side.proj", "norm": "l4.side.norm", "from": 28}
    assert [first["mlp"][key] for key in ("experts", "top", "ff", "limit", "scores")] == [9, 3, 50, 1.5, "softmax_chosen"] and fourth["mlp"] is None
    # a repeated pass begins with nothing but the stream
    assert [run["layer"] for run in program["runs"]] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4] and not any(run["add_embedding"] for run in program["runs"])
    assert sum(run["add_embedding"] for run in looped_runs(5, config["loop"])) == 2
    shapes = tensor_shapes(config)
    assert shapes["l0.mix.uq"] == (5 * 26, 21) and shapes["l0.mix.dkv"] == (49, 90) and shapes["l0.mix.dkv.norm"] == (43,) and shapes["l0.mix.dq.norm"] == (21,)
    assert shapes["l1.mix.w1"] == (5, 90) and shapes["l1.mix.w2"] == (66, 5) and shapes["l1.mix.a.b"] == (66,) and shapes["l1.mix.norm"] == (66,)
    assert shapes["l3.canon1"] == (90, 4) and shapes["side.embed"] == (203, 35) and shapes["l3.side.proj"] == (90, 7) and "l0.norm2" not in shapes
    for wrong, message in (({"type": "other"}, "unknown layer type"), ({"mlp": {"kind": "dense"}}, "unknown feed-forward"),
                           ({"mixer": config["layers"][0]["mixer"] | {"rot_dim": 4}}, "whole rotated part")):
        with pytest.raises(ValueError, match=message):
            family_of(config).layer_program(config | {"layers": [config["layers"][0] | wrong]})


def test_sizes_that_only_the_tensors_tell(tmp_path):
    from safetensors.torch import save_file
    config = case.CASES["ones"]
    plain = json.loads(json.dumps(config))
    del plain["layers"][1]["mixer"]["decay_rank"]
    (tmp_path / "config.json").write_text(json.dumps(plain))
    save_file({name: torch.zeros(shape, dtype=torch.bfloat16) for name, shape in tensor_shapes(config).items()}, tmp_path / "model.safetensors")
    assert load_config(tmp_path) == config


@pytest.mark.parametrize("name", sorted(case.CASES))
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_buffer_table_and_recipes(name, dtype, plan_dir):
    config = case.CASES[name]
    library = PlanLibrary(emit_plan(config, plan_dir, phase="ragged", slots=3, capacity=64, num_blocks=9, max_rows=32, dtype=dtype))
    assert library.info.phase == RAGGED
    tensors = case.weights(config)
    loaded = load_weights(TensorCheckpoint(tensors), library, device="cpu")    # element counts are checked inside
    up = lambda count, unit=8: -(-count // unit) * unit
    width, side = config["width"], config["token_side"]["dim"]
    assert torch.equal(loaded["side.embed"].float(), tensors["side.embed"])
    for index, item in enumerate(config["layers"]):
        p, mixer = f"l{index}.", item["mixer"]
        heads, dim = mixer["heads"], mixer["dim"]
        assert torch.equal(loaded[p + "conv"].reshape(-1, width), tensors[p + "canon1"].T)
        assert torch.equal(loaded[p + "side.proj"].float().reshape(width, up(side))[:, :side], tensors[p + "side.proj"])
        stacked = loaded[p + "in.weight"].float().reshape(-1, up(width))
        assert not stacked[:, width:].any()
        stacked = stacked[:, :width]
        if item["type"] == "general_delta":
            rank, all_heads = mixer["decay_rank"], heads * dim
            assert torch.equal(stacked[:rank], tensors[p + "mix.w1"]) and not stacked[rank:up(rank)].any()
            assert torch.equal(stacked[up(rank):], torch.cat([tensors[p + "mix." + part] for part in ("r", "k", "v", "a", "g")]))
            bias = loaded[p + "in.bias"]
            assert torch.equal(bias[up(rank) + 3 * all_heads:][:all_heads], tensors[p + "mix.a.b"]) and bias.count_nonzero() <= all_heads
            assert torch.equal(loaded[p + "decay_up.weight"].float().reshape(all_heads, up(rank))[:, :rank], tensors[p + "mix.w2"])
            continue
        rank, rot, vdim, q_rank = (mixer[key] for key in ("kv_rank", "rot_dim", "vdim", "q_rank"))
        # entries that turn together are neighbours: in the shared key part and behind every head's others in the queries
        order = torch.arange(rot) if item["type"] == "latent_attention" else torch.arange(rot).reshape(2, -1).T.reshape(-1)
        assert torch.equal(stacked[:q_rank], tensors[p + "mix.dq"]) and not stacked[q_rank:up(q_rank)].any()
        assert torch.equal(stacked[up(q_rank):up(q_rank) + rank], tensors[p + "mix.dkv"][:rank])
        assert torch.equal(stacked[up(q_rank) + rank:], tensors[p + "mix.dkv"][rank:][order])
        step = up(dim) + up(rot)
        query = loaded[p + "query_up.weight"].float().reshape(heads, step, up(q_rank))[..., :q_rank]
        original = tensors[p + "mix.uq"].reshape(heads, dim + rot, q_rank)
        assert torch.equal(query[:, :dim], original[:, :dim]) and torch.equal(query[:, up(dim):up(dim) + rot], original[:, dim:][:, order])
        assert not query[:, dim:up(dim)].any() and not query[:, up(dim) + rot:].any()
        # a query against latent rows: the head's key matrix transposed, the rotated part as it is
        row = up(rank + rot)
        turned = loaded[p + "key_up.weight"].float().reshape(heads, row, step)
        assert torch.equal(turned[heads - 1, :rank, :dim], tensors[p + "mix.uk"].reshape(heads, dim, rank)[heads - 1].T)
        assert torch.equal(turned[0, rank:rank + rot, up(dim):up(dim) + rot], torch.eye(rot)) and turned[0, rank:].sum() == rot and not turned[0, :rank, dim:].any()
        values = loaded[p + "value_up.weight"].float().reshape(heads * vdim, row)
        assert torch.equal(values[:, :rank], tensors[p + "mix.uv"]) and not values[:, rank:].any()
        if dtype == "bf16":
            key = up(up(dim) + rot, 16)
            expanded = loaded[p + "expand.weight"].float().reshape(-1, row)
            keys, rest = expanded[:heads * key].reshape(heads, key, row), expanded[heads * key:].reshape(heads, -1, row)
            assert torch.equal(keys[:, :dim, :rank].reshape(-1, rank), tensors[p + "mix.uk"]) and torch.equal(keys[heads - 1, up(dim):up(dim) + rot, rank:rank + rot], torch.eye(rot))
            assert torch.equal(rest[:, :vdim, :rank].reshape(-1, rank), tensors[p + "mix.uv"]) and not rest[:, :, rank:].any()
    state = allocate_ragged_state(library, "cpu")
    runs, taps = oracle.order(config), config["canon"]["taps"]
    for number, index in enumerate(runs):          # every pass has its own
        mixer = config["layers"][index]["mixer"]
        if config["layers"][index]["type"] == "general_delta":
            assert state[f"delta.{number}"].numel() == 3 * mixer["heads"] * mixer["dim"] * up(mixer["dim"], 4)
        else:
            assert state[f"kv_pool.latent.{number}"].numel() == 9 * 16 * up(mixer["kv_rank"] + mixer["rot_dim"], 16)
        assert (f"history.{number}" in state) == (taps > 1)
        if taps > 1:
            assert state[f"history.{number}"].numel() == 3 * (taps - 1) * width


def test_rotary_tables_with_a_stretched_length():
    for rot in ({"base": 10000.0, "dims": 32}, {"base": 500.0, "dims": 12, "scaling": case.stretch()},
                {"base": 10000.0, "dims": 64, "scaling": case.stretch(8.0, 512, 32.0, 1.0)}, {"base": 10000.0, "dims": 8, "scaling": case.stretch(2.0, 4, 8.0, 7.0)}):
        table = rotary_pairs(rot["base"], rot["dims"], 50, yarn=rot.get("scaling"))
        turn, size = oracle.frequencies(rot)
        angles = torch.arange(50, dtype=torch.float64)[:, None] * torch.tensor(turn, dtype=torch.float64)
        assert torch.allclose(table[..., 0].double(), size * angles.cos(), atol=1e-6) and torch.allclose(table[..., 1].double(), size * angles.sin(), atol=1e-6)


@pytest.mark.parametrize("break_it, message", [
    (lambda m: m["layers"][0]["mixer"].update(vdim=300), "head sizes"),
    (lambda m: m["layers"][0]["mixer"].update(dim=253), "head sizes"),
    (lambda m: m["layers"][0]["mixer"].update(rank=1020), "1..1024 columns"),
    (lambda m: m["layers"][0]["mixer"].update(q_rank=0), "row of their own"),
    (lambda m: m["layers"][4]["mixer"]["rotary"]["yarn"].update(fast=0), "length scaling"),
    (lambda m: m["layers"][1]["mixer"].update(vdim=10), "one size per head"),
    (lambda m: m["layers"][1]["mixer"].update(decay_rank=0), "decays' row"),
    (lambda m: m["layers"][1]["mixer"].update(decay_scale=4.5), "factor of e.4 per token"),
    (lambda m: m["layers"][0]["side"].update({"from": 30}), "second embedding"),
    (lambda m: m["layers"][0]["mlp"].update(shared={"ff": 8, "limit": 1.0}), "no shared expert"),
    (lambda m: m["layers"][0]["mlp"].update(groups={"count": 3, "keep": 1}), "logits alone"),
    (lambda m: m["layers"][0].update(norm_at="output"), "read one norm"),
    (lambda m: m["runs"][4].update(add_embedding=True), "embedding added"),
    (lambda m: m.update(norm_groups=4), "equal runs"),
    (lambda m: m.update(taps=17), "1..16 taps"),
    (lambda m: m.update(streams=2), "parallel layers have one stream"),
    (lambda m: m.update(form="sequential"), "built for parallel layers"),
])
def test_unsupported_programs_are_refused(break_it, message, plan_dir, capfd):
    so = emit_plan(case.CASES["odd"], plan_dir, phase="ragged", slots=2, capacity=32, num_blocks=5, max_rows=16)
    document = json.loads((so.parent / (so.name + ".plan.json")).read_text())
    break_it(document["model"])
    broken = so.parent / f"tilemega_b200_refused_benarax_{abs(hash((message, str(document)))) % 10 ** 8}.so"
    shutil.copyfile(so, broken)
    (so.parent / (broken.name + ".plan.json")).write_text(json.dumps(document))
    with pytest.raises(RuntimeError, match=message):
        PlanLibrary(broken)


def test_recipes():
    matrix = torch.arange(1.0, 25.0).reshape(6, 4)
    grown = per_head({"kind": "append_identity", "heads": 2, "size": 2}, matrix)
    assert grown.shape == (10, 6) and torch.equal(grown[:3, :4], matrix[:3]) and torch.equal(grown[5:8, :4], matrix[3:])
    assert torch.equal(grown[8:, 4:], torch.eye(2)) and not grown[:3, 4:].any() and not grown[3:5, :4].any()
    wide = torch.arange(1.0, 11.0).reshape(10, 1)
    tail = lambda layout: per_head({"kind": "rotary_tail", "heads": 2, "dims": 4, "layout": layout, "lead": 2, "rows": 7}, wide)[:, 0].tolist()
    assert tail("pairs") == [1, 0, 2, 3, 4, 5, 0, 6, 0, 7, 8, 9, 10, 0] and tail("halves") == [1, 0, 2, 4, 3, 5, 0, 6, 0, 7, 9, 8, 10, 0]
    assert pack({"kind": "pad_vector", "before": 2, "behind": 1, "source": "x"}, lambda name: torch.tensor([5.0, 6.0])).tolist() == [0, 0, 5, 6, 0]
    for recipe in ({"kind": "append_identity", "heads": 2, "size": 0}, {"kind": "rotary_tail", "heads": 2, "dims": 2, "layout": "other", "lead": 3, "rows": 5},
                   {"kind": "rotary_tail", "heads": 2, "dims": 3, "layout": "pairs", "lead": 3, "rows": 6},
                   {"kind": "rotary_tail", "heads": 2, "dims": 2, "layout": "pairs", "lead": 0, "rows": 6}):
        with pytest.raises(ValueError):
            per_head(recipe, matrix)


def test_coded_routers_rest_on_no_close_call():
    for name in ("odd", "wide", "crowd"):
        config = case.CASES[name]
        tensors, ids, gaps = case.weights(config, coded=True), case.tokens(config, 40), []
        original = oracle.route

        def watched(z, top):
            ranked = z.sort(descending=True).values
            if top < len(z):
                gaps.append(float(ranked[top - 1] - ranked[top]))
            return original(z, top)

        oracle.route = watched
        try:
            case.truth(config, tensors, ids)
        finally:
            oracle.route = original
        assert min(gaps) > 0.03, (name, min(gaps))


# ---- the plain forward's mechanisms --------------------------------------------------------------------------------------
def draws(*shapes):
    generator = torch.Generator().manual_seed(6)
    return [torch.randn(*shape, generator=generator, dtype=torch.float64) for shape in shapes]


def test_plain_grouped_norm():
    x, weight = draws((5, 12), (12,))
    got = oracle.grouped_norm(x, weight, 3, 1e-2)
    for t in range(5):
        for c in range(12):
            part = x[t, c // 4 * 4:c // 4 * 4 + 4]
            assert float(got[t, c]) == pytest.approx(float(x[t, c] * weight[c]) / math.sqrt(float((part ** 2).sum()) / 4 + 1e-2))


def test_plain_convolution_against_the_definition():
    h, kernel = draws((7, 3), (3, 4))
    got = oracle.short_convolution(h, kernel)
    for t in range(7):
        for c in range(3):
            want = sum(float(kernel[c, j] * h[t - 4 + 1 + j, c]) for j in range(4) if t - 4 + 1 + j >= 0)
            assert float(got[t, c]) == pytest.approx(want)


def test_plain_latent_mixer_against_latent_rows_themselves():
    """Expanded keys and values, and queries and sums against the latent rows with the rotated part behind them, are the same."""
    spec = {"heads": 3, "dim": 4, "rot_dim": 2, "vdim": 5, "kv_rank": 7, "q_rank": 6, "scale": 0.3, "rot": {"base": 50.0, "dims": 2}}
    h, dq, dq_norm, uq, dkv, norm, uk, uv, o = draws((9, 10), (6, 10), (6,), (18, 6), (9, 10), (7,), (12, 7), (15, 7), (10, 15))
    named = {"dq": dq, "dq.norm": dq_norm, "uq": uq, "dkv": dkv, "dkv.norm": norm, "uk": uk, "uv": uv, "o": o}
    got = oracle.latent_mixer(h, torch.arange(9), spec, named.__getitem__, 1e-4, True)
    unit = lambda x: x / (x.pow(2).mean(-1, keepdim=True) + 1e-4).sqrt()
    q = ((unit(h @ dq.T) * dq_norm) @ uq.T).reshape(9, 3, 6)
    c = unit((h @ dkv.T)[:, :7]) * norm

    def turn(x, t):                                              # one pair: angle t
        return torch.stack((x[..., 0] * math.cos(t) - x[..., 1] * math.sin(t), x[..., 1] * math.cos(t) + x[..., 0] * math.sin(t)), -1)

    rows = torch.stack([torch.cat((c[t], turn((h @ dkv.T)[t, 7:], t))) for t in range(9)])
    out = torch.zeros(9, 15, dtype=torch.float64)
    for i in range(9):
        for head in range(3):
            lookup = torch.cat((q[i, head, :4] @ uk.reshape(3, 4, 7)[head], turn(q[i, head, 4:], i)))
            weight = torch.softmax(0.3 * rows[:i + 1] @ lookup, 0)
            out[i, 5 * head:5 * head + 5] = uv.reshape(3, 5, 7)[head] @ (weight @ c[:i + 1])
    assert torch.allclose(got, out @ o.T)


def test_plain_rotations_and_stretched_lengths():
    (q,) = draws((1, 1, 6))
    for neighbours in (True, False):
        turned = oracle.rotate(q, torch.tensor([9]), {"base": 50.0, "dims": 6}, neighbours)
        for i in range(3):
            a, (x, y) = 9 * 50.0 ** (-2 * i / 6), ((2 * i, 2 * i + 1) if neighbours else (i, i + 3))
            u, v = float(q[0, 0, x]), float(q[0, 0, y])
            assert float(turned[0, 0, x]) == pytest.approx(u * math.cos(a) - v * math.sin(a))
            assert float(turned[0, 0, y]) == pytest.approx(v * math.cos(a) + u * math.sin(a))
    turn, size = oracle.frequencies({"base": 10000.0, "dims": 64, "scaling": case.stretch(4.0, 4096, 32.0, 1.0)})
    assert size == pytest.approx(0.1 * math.log(4) + 1) and turn[0] == 1.0
    assert turn[31] == pytest.approx(10000.0 ** (-62 / 64) / 4)      # a pair that never turns once over the original length
    fast, slow = math.floor(64 * math.log(4096 / (64 * math.pi)) / (2 * math.log(10000.0))), math.ceil(64 * math.log(4096 / (2 * math.pi)) / (2 * math.log(10000.0)))
    middle = (fast + slow) // 2
    ramp = (middle - fast) / (slow - fast)
    assert turn[middle] == pytest.approx(10000.0 ** (-2 * middle / 64) * (ramp / 4 + 1 - ramp))


def test_plain_delta_rule_against_matrices():
    r, k, v, z, a = draws((6, 4), (6, 4), (6, 4), (6, 4), (6, 4))
    w, a = oracle.decay_of(z), torch.sigmoid(a)
    assert float(w.min()) > math.exp(-math.exp(-0.5)) and float(w.max()) < 1.0
    got = oracle.delta_recurrence(r, k, v, w, a)
    state = torch.zeros(4, 4, dtype=torch.float64)
    for t in range(6):
        u = k[t] / math.sqrt(float(k[t] @ k[t]) + 1e-6)
        state = (torch.diag(w[t]) - torch.outer(a[t] * u, u)) @ state + torch.outer(k[t], v[t])
        assert torch.allclose(got[t], state.T @ r[t])


def test_plain_routing_weighs_among_the_chosen():
    z = torch.tensor([0.1, 2.0, -1.0, 2.0, 1.5], dtype=torch.float64)
    chosen, weights = oracle.route(z, 3)
    assert chosen == [1, 3, 4] and torch.allclose(weights, torch.softmax(torch.tensor([2.0, 2.0, 1.5], dtype=torch.float64), 0))


def test_plain_side_input_and_unit():
    x, e, gate, proj, norm = draws((3, 6), (3, 2), (2, 6), (6, 2), (6,))
    got = oracle.side_input(x, e, {"gate": gate, "proj": proj, "norm": norm}.__getitem__, 1e-3)
    z = gate @ x[1]
    g = torch.tensor([0.5 * t * (1 + math.tanh(math.sqrt(2 / math.pi) * (t + 0.044715 * t ** 3))) for t in z.tolist()], dtype=torch.float64)
    y = proj @ (g * e[1])
    assert torch.allclose(got[1], y / math.sqrt(float((y * y).mean()) + 1e-3) * norm)
    h, gate, up, down = draws((30, 8), (5, 8), (5, 8), (8, 5))
    got, want = oracle.clipped_unit(h, 0.7, {"gate": gate, "up": up, "down": down}.__getitem__), torch.zeros(5, dtype=torch.float64)
    for j in range(5):
        g, u = min(float(gate[j] @ h[3]), 0.7), max(-0.7, min(0.7, float(up[j] @ h[3])))
        want[j] = g / (1 + math.exp(-1.702 * g)) * (u + 1)
    assert torch.allclose(got[3], down @ want)
