"""Faults that random weights would hide in a Mozidra-shaped model: a window one token off, a far key, a sink left out or
scaled, a norm per head, an angle of the wrong pair, values mixed with the wrong layer's, a stream matrix read the wrong way
round, a ruled-out expert. The weights are made so that each shows; wrong variants run in the plain forward only."""
import copy

import pytest
import torch

import mozidra_case as case
from oracle import mozidra_oracle as oracle
from test_gpu_ragged import DTYPES, executor, run_cut
from tilemega_b200.serving.ragged import Portion

pytestmark = pytest.mark.gpu
MARK = 7          # the token that stands out
KINDS = ["attention", "latent"]


def bf16(tensors):
    return {name: tensor.to(torch.bfloat16).float() for name, tensor in tensors.items()}


def one_layer(kind, window, heads=4, kv_heads=2, dim=24, vdim=18, rank=20, rot=10, scale=0.5, mlp=None, streams=2, width=40):
    if kind == "latent":
        return case.model(width, 61, [case.latent(heads, dim, vdim, rank, window, mlp, scale)], streams)
    return case.model(width, 61, [case.grouped(heads, kv_heads, dim, vdim, rot, window, mlp, scale=scale)], streams)


def standing_out(kind, window, **sizes):
    """One layer in which every query points along one (unrotated) direction and only MARK's key lies along it: wherever
    MARK is seen it takes nearly all of the weight."""
    config = one_layer(kind, window, **sizes)
    spec, tensors = config["layers"][0]["mixer"], case.weights(config, seed=3)
    dim = spec["dim"]
    tensors["embed"][:, 0] = 0.0
    tensors["embed"][:, 1] = 1.0                                 # every token
    tensors["embed"][MARK, 2:] *= 0.1
    tensors["embed"][MARK, 0] = 4.0                              # alone in column 0
    tensors["l0.mix.q"].mul_(0.05)
    tensors["l0.mix.q"][dim - 1::dim, 1] = 3.0
    if kind == "latent":
        tensors["l0.mix.dkv"][0] = 0.0
        tensors["l0.mix.dkv"][0, 0] = 4.0                        # MARK's latent row alone has an entry 0
        tensors["l0.mix.uk"][dim - 1::dim] = 0.0
        tensors["l0.mix.uk"][dim - 1::dim, 0] = 3.0
        tensors["l0.mix.uv"][:, 0] = torch.linspace(-1, 1, len(tensors["l0.mix.uv"]))
    else:
        tensors["l0.mix.q.b"].mul_(0.05)
        tensors["l0.mix.k.b"][dim - 1::dim] = 0.0
        tensors["l0.mix.k"][dim - 1::dim] = 0.0
        tensors["l0.mix.k"][dim - 1::dim, 0] = 2.0
        tensors["l0.mix.v"][:, 0] = torch.linspace(-1, 1, len(tensors["l0.mix.v"]))
    return config, bf16(tensors)


def marked(config, length, places, seed):
    ids = [token if token != MARK else MARK + 1 for token in case.tokens(config, length, seed=seed)]
    for place in places:
        ids[place] = MARK
    return ids


def changed(config, **mask):
    other = copy.deepcopy(config)
    other["layers"][0]["mixer"]["mask"].update(mask)
    return other


def altered(name, wrong, config, tensors, ids):
    """The plain forward's logits with one of its functions replaced."""
    original = getattr(oracle, name)
    setattr(oracle, name, wrong(original))
    try:
        return case.truth(config, tensors, ids)[0]
    finally:
        setattr(oracle, name, original)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 63, 64, 65, 128])
def test_window_edges(window, kind, dtype, plan_dir):
    """MARK at block borders, just inside and just outside the window of later positions: each position's logits in one
    prompt, in portions and decoded are the plain forward's, and a window that is one off would show."""
    config, tensors = standing_out(kind, window, rank=20 if window % 2 else 90)   # (long portions expand wide rows only)
    with executor(config, tensors, plan_dir, dtype, capacity=256) as ex:
        for place in (0, 1, 15, 16, 64):
            ids = marked(config, place + window + 12, [place], seed=place)
            want = case.truth(config, tensors, ids)[0]
            for size in (window + 1, window - 1):
                if size > 0:
                    assert case.error(case.truth(changed(config, size=size), tensors, ids)[0], want) > 5 * case.TOLERANCE[dtype]
            for cuts in ([len(ids)], [place + 1, 1], [place + window, 2], [5, 2, 33, 1]):
                assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], (place, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind, sizes", [("attention", dict(dim=40, vdim=56)), ("latent", dict(dim=40, vdim=56, rank=30)),
                                         ("latent", dict(dim=16, vdim=16, rank=200, heads=40)), ("latent", dict(dim=16, vdim=24, rank=450, heads=70))])
def test_a_far_key_among_a_thousand(kind, sizes, dtype, plan_dir):
    """MARK a thousand positions back, seen and no longer seen, by rows of a prompt and by decoded tokens whose window is
    cut over several CTAs, beside other sequences."""
    config, tensors = standing_out(kind, 1100, **sizes)
    ids = marked(config, 1230, [70], seed=4)
    want = case.truth(config, tensors, ids)[0]
    blind = case.truth(config, tensors, [8 if token == MARK else token for token in ids])[0]
    assert case.error(blind[1000:1169], want[1000:1169]) > 5 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype, slots=3, capacity=1264, max_rows=1264, max_wanted=1264) as ex:
        for cuts in ([1230], [1100, 130], [600, 500, 2, 3, 125]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts
        slots = [ex.open() for _ in range(3)]
        starts = [1160, 300, 1120]                               # the first leaves MARK behind while it decodes
        for slot, start in zip(slots, starts):
            ex.run([Portion(slot, ids[:start])])
        for turn in range(25):
            got = ex.run([Portion(slot, [ids[start + turn]], [0]) for slot, start in zip(slots, starts)])
            assert case.error(got, want[[start + turn for start in starts]]) < case.TOLERANCE[dtype], turn


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", KINDS)
def test_first_tokens_rest_on_the_sinks(kind, dtype, plan_dir):
    """Sinks high, near zero and far below: without them, with the scores' scale on them, with another head's, or counted
    twice, the first positions' outputs would differ."""
    config = one_layer(kind, 20, heads=3, kv_heads=1, dim=16, vdim=12, scale=0.3)
    tensors = case.weights(config, seed=8)
    tensors["l0.mix.sink"] = torch.tensor([4.0, 1.0, -3.0])
    tensors["l0.mix.o"] *= 3.0
    tensors = bf16(tensors)
    ids = case.tokens(config, 40)
    want = case.truth(config, tensors, ids)[0]
    for wrong in (lambda f: lambda score, seen, sink: torch.softmax(score.masked_fill(~seen, float("-inf")), -1),
                  lambda f: lambda score, seen, sink: f(score, seen, 0.3 * sink),
                  lambda f: lambda score, seen, sink: f(score, seen, sink + 0.693147),
                  lambda f: lambda score, seen, sink: f(score, seen, -sink)):
        assert case.error(altered("softmax_with_sink", wrong, config, tensors, ids)[:4], want[:4]) > 1.5 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([40], [1], [2], [1, 39], [3, 1]):
            got = run_cut(ex, ids, cuts)
            assert case.error(got, want) < case.TOLERANCE[dtype] and case.error(got[:2], want[:2]) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", KINDS)
def test_scores_far_from_zero(kind, dtype, plan_dir):
    """Scores in the hundreds: all far below the sink, which then takes everything, and a sink of hundreds on either side."""
    config = one_layer(kind, 90, heads=4, kv_heads=2, dim=16, vdim=16, rank=24, rot=4, scale=-20.0)
    tensors = case.weights(config, seed=9)
    tensors["embed"][:, 1] = 3.0
    tensors["l0.mix.q"][15::16, 1] = 2.0
    if kind == "latent":
        tensors["l0.mix.dkv"][3, 1] = 5.0
        tensors["l0.mix.uk"][15::16, 3] = 2.0
    else:
        tensors["l0.mix.k"][15::16, 1] = 2.0                     # q . k > 0 throughout
    for sink in ([0.0, 1.0, -1.0, 3.0], [200.0, 0.0, 90.0, 4.0]):
        tensors["l0.mix.sink"] = torch.tensor(sink)
        rounded = bf16(tensors)
        ids = case.tokens(config, 100)
        want = case.truth(config, rounded, ids)[0]
        assert torch.isfinite(want).all()
        with executor(config, rounded, plan_dir, dtype) as ex:
            for cuts in ([100], [60, 1]):
                got = run_cut(ex, ids, cuts)
                assert torch.isfinite(got).all() and case.error(got, want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_over_all_heads_together(dtype, plan_dir):
    """Heads of very unequal size: a norm per head would bring them to the same size."""
    config = one_layer("attention", 30, heads=6, kv_heads=3, dim=16, vdim=8, rot=8, scale=0.7, width=48)
    tensors = case.weights(config, seed=12)
    for part, heads, base in (("q", 6, 2.0), ("k", 3, 0.33)):
        for head in range(heads):
            for name in (f"l0.mix.{part}", f"l0.mix.{part}.b"):
                tensors[name][16 * head:16 * head + 16] *= base ** (head - heads // 2)
    tensors = bf16(tensors)
    ids = case.tokens(config, 70)
    want = case.truth(config, tensors, ids)[0]
    wrong = lambda f: lambda x, eps: f(x.reshape(len(x), -1, 16), eps).reshape(x.shape) if x.shape[-1] in (96,) else f(x, eps)
    assert case.error(altered("rms", wrong, config, tensors, ids), want) > 2 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([70], [33, 1], [2]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
def test_neighbours_turn_together_at_far_positions(dtype, plan_dir):
    """Rotations of part of a head and of all of it, thousands of positions from the start: angles and distances stay exact,
    and halves in place of neighbours would show."""
    config = case.model(24, 40, [case.grouped(2, 1, 16, 12, 16, 50, base=300.0, scale=0.6), case.grouped(2, 2, 12, 6, 6, 30, base=90.0, scale=0.8)])
    tensors, ids = case.weights(config), case.tokens(config, 2000)
    want = case.truth(config, tensors, ids)[0]

    def halves(f):
        def turned(x, positions, base, dims):
            order = torch.arange(x.shape[-1])
            order[:dims] = torch.arange(dims).reshape(2, -1).T.reshape(-1)
            return f(x[..., order], positions, base, dims)
        return turned

    assert case.error(altered("rotate_pairs", halves, config, tensors, ids[:60]), want[:60]) > 3 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype, slots=1, capacity=2000, max_rows=1000) as ex:
        slot = ex.open()
        out = [ex.run([Portion(slot, ids[at:at + 650], [649])]) for at in (0, 650, 1300)]
        for at in range(1950, 2000):
            out.append(ex.run([Portion(slot, [ids[at]], [0])]))
    assert case.error(torch.cat(out), want[[649, 1299, 1949] + list(range(1950, 2000))]) < 2 * case.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_values_are_mixed_with_the_first_mixing_layer(dtype, plan_dir):
    """Layers of which the second and the last two mix: with the second's values, not the first layer's nor the one before;
    shares of 0 and of 1."""
    layers = [case.grouped(2, 2, 16, 12, 8, 20, mixing=index in (1, 3, 4)) for index in range(5)]
    config = case.model(48, 61, layers)
    tensors = case.weights(config, seed=14)
    for index, share in ((3, 1.0), (4, 0.25)):
        tensors[f"l{index}.mix.vmix"] = torch.tensor(share)
    tensors = bf16(tensors)
    ids = case.tokens(config, 90)
    want = case.truth(config, tensors, ids)[0]
    for mixing in ((), (0, 3, 4), (3, 4), (1, 3)):
        other = copy.deepcopy(config)
        for index, layer in enumerate(other["layers"]):
            layer["mixer"]["v_mix"] = index in mixing
        assert case.error(case.truth(other, tensors, ids)[0], want) > 2 * case.TOLERANCE[dtype], mixing
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([90], [1], [33, 2, 1], [2]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts
        # two sequences in one step: each with its own rows of the first layer's values
        a, b = ex.open(), ex.open()
        ex.run([Portion(a, ids[:30]), Portion(b, ids[:70])])
        got = ex.run([Portion(b, [ids[70]], [0]), Portion(a, ids[30:50], [0, 19])])
        assert case.error(got, want[[70, 30, 49]]) < case.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 7, 16])
@pytest.mark.parametrize("width", [48, 50])
def test_streams(streams, width, dtype, plan_dir):
    """Stream matrices far from symmetric, streams of unequal weight: read from the wrong side, or one stream after the other
    instead of all from the old ones, would show. Widths with and without the vectorised form."""
    config = case.model(width, 61, [case.latent(2, 8, 12, 10, 9, case.moe(4, 2, 24)), case.grouped(2, 1, 8, 12, 4, 9),
                                    case.latent(3, 8, 12, 16, 9, case.moe(2, 1, 24))], streams)
    tensors = case.weights_for(config, dtype, seed=streams)
    generator = torch.Generator().manual_seed(streams)
    for name, tensor in tensors.items():
        if name.split(".")[-1] == "mix" and ".hc" in name:
            tensor.copy_(0.5 * torch.eye(streams) + torch.randn(tensor.shape, generator=generator) * streams ** -0.5)
        elif ".hc" in name:
            tensor.copy_(torch.rand(tensor.shape, generator=generator) + 0.1)
    tensors = bf16(tensors)
    ids = case.tokens(config, 70)
    want, kept = case.truth(config, tensors, ids)
    if streams > 1:
        other = altered("distribute", lambda f: lambda x, mix, out, y: f(x, mix.T, out, y), config, tensors, ids)
        assert case.error(other, want) > case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype, write_residuals=True) as ex:
        assert case.error(run_cut(ex, ids, [70]), want) < case.TOLERANCE[dtype]
        for got, expected in zip(ex.residuals(len(ids)), kept):
            assert case.error(got, expected) < case.TOLERANCE[dtype]
        assert case.error(run_cut(ex, ids, [20, 1]), want) < case.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts, top, groups, keep", [(24, 1, 4, 1), (24, 2, 24, 3), (24, 5, 1, 1), (200, 5, 8, 3), (12, 4, 3, 1), (3, 3, 1, 1), (300, 6, 20, 4),
                                                        (320, 3, 320, 5)])
def test_routing(experts, top, groups, keep, dtype, plan_dir):
    """Steps of 1 to 700 rows, around the size at which routing changes its form and at which tiles grow; corrections that
    lift experts of low score and rule out ones of high score, so that weights, ranks and groups all differ."""
    if dtype == "bf16" and experts == 300:
        pytest.skip("three hundred levels lie too close together for 16 bits")
    config = case.model(340, 130, [case.latent(2, 16, 16, 8, 10, case.moe(experts, top, 40, groups, keep))])
    tensors = case.weights_for(config, dtype, seed=7)
    ids = case.tokens(config, 700)
    want = case.truth(config, tensors, ids)[0]
    if keep < groups < experts and top > 1 and dtype == "f32":      # without groups
        other = copy.deepcopy(config)
        other["layers"][0]["mlp"]["router"]["groups"] = {"count": 1, "keep": 1}
        assert case.error(case.truth(other, tensors, ids[:60])[0], want[:60]) > 1000 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype, slots=1, capacity=704, max_rows=704, max_wanted=704) as ex:
        for cuts in ([700], [63, 64, 65, 128, 129, 251], [1, 2, 7, 33, 300, 357], [690, 1]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
def test_limits_of_experts_and_of_the_shared_one(dtype, plan_dir):
    """Activations well beyond both limits, which differ: a limit left out, or the other's, would show."""
    config = case.model(64, 90, [case.latent(2, 16, 16, 24, 20, case.moe(4, 2, 32, limit=0.9, shared=48, shared_limit=2.5))])
    tensors, ids = case.weights_for(config, dtype, seed=2), case.tokens(config, 75)
    for name, tensor in tensors.items():
        if name.endswith((".gate", ".up")):
            tensor *= 3.0
    tensors = bf16(tensors)
    want = case.truth(config, tensors, ids)[0]
    for part, limit in (("expert", 2.5), ("shared", 0.9), ("shared", 50.0)):
        other = copy.deepcopy(config)
        other["layers"][0]["mlp"][part]["limit"] = limit
        assert case.error(case.truth(other, tensors, ids)[0], want) > 2 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([75], [63, 1], [64, 2], [65, 3]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


def test_many_sequences_decode_together(plan_dir):
    """Batches of 1 to 70 decoded tokens (routing inside one kernel up to 64 rows) give each sequence what it gets alone."""
    config = case.CASES["wide"]
    tensors = case.weights(config, coded=True)
    ids = [case.tokens(config, 24, seed=100 + index) for index in range(70)]
    wanted = [case.truth(config, tensors, sequence)[0] for sequence in ids]
    with executor(config, tensors, plan_dir, "bf16", slots=70, capacity=32, max_rows=1120) as ex:
        slots = [ex.open() for _ in ids]
        ex.run([Portion(slot, sequence[:16]) for slot, sequence in zip(slots, ids)])
        for turn, count in enumerate((70, 64, 65, 33, 16, 3, 1, 70)):
            done = [16 + sum(1 for c in (70, 64, 65, 33, 16, 3, 1)[:turn] if index < c) for index in range(70)]
            got = ex.run([Portion(slots[index], [ids[index][done[index]]], [0]) for index in range(count)])
            want = torch.stack([wanted[index][done[index]] for index in range(count)])
            assert case.error(got, want) < case.TOLERANCE["bf16"], count
