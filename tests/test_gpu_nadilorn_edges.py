"""Faults that random weights would hide in a Nadilorn-shaped model: a window one token off, a far key, the null key left
out, a norm per head instead of over all heads, an angle that is not scaled, a score on the wrong side of an expert, a
routing table that overflows. The weights are made so that each shows; wrong variants run in the plain forward only."""
import copy

import pytest
import torch

import nadilorn_case as case
from oracle import nadilorn_oracle as oracle
from test_gpu_ragged import DTYPES, executor, run_cut
from tilemega_b200.serving.ragged import Portion

pytestmark = pytest.mark.gpu
MARK = 7          # the token that stands out


def bf16(tensors):
    return {name: tensor.to(torch.bfloat16).float() for name, tensor in tensors.items()}


def standing_out(window, dim=24, vdim=18, rot=10, heads=4, kv_heads=2):
    """One layer in which every query points along an unrotated direction and only MARK's key lies along it: wherever MARK
    is seen it takes nearly all of the weight."""
    config = case.model(40, 61, [case.layer(heads, kv_heads, dim, vdim, rot, window, scale=0.5)])
    tensors = case.weights(config, seed=3)
    q, k = tensors["l0.mix.q"], tensors["l0.mix.k"]
    q.mul_(0.05)
    k[dim - 1::dim] = 0.0                                        # nothing of the other tokens' keys
    tensors["embed"][:, 0] = 0.0
    tensors["embed"][:, 1] = 1.0                                 # every token
    tensors["embed"][MARK, 2:] *= 0.1
    tensors["embed"][MARK, 0] = 4.0                              # alone in column 0
    q[dim - 1::dim, 1] = 3.0
    k[dim - 1::dim, 0] = 2.0
    tensors["l0.mix.v"][:, 0] = torch.linspace(-1, 1, kv_heads * vdim)
    return config, bf16(tensors)


def changed(config, **mask):
    other = copy.deepcopy(config)
    other["layers"][0]["mixer"]["mask"].update(mask)
    return other


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 63, 64, 65, 128])
def test_window_edges(window, dtype, plan_dir):
    """MARK at block borders, just inside and just outside the window of later positions: each position's logits in one
    prompt, in portions and decoded are the plain forward's, and a window that is one off would show."""
    config, tensors = standing_out(window)
    with executor(config, tensors, plan_dir, dtype, capacity=256) as ex:
        for place in (0, 1, 15, 16, 64):
            ids = [token if token != MARK else MARK + 1 for token in case.tokens(config, place + window + 12, seed=place)]
            ids[place] = MARK
            want = case.truth(config, tensors, ids)[0]
            for size in (window + 1, window - 1):
                if size > 0:
                    assert case.error(case.truth(changed(config, size=size), tensors, ids)[0], want) > 5 * case.TOLERANCE[dtype]
            for cuts in ([len(ids)], [place + 1, 1], [place + window, 2], [5, 2, 33, 1]):
                assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], (place, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_among_a_thousand(dtype, plan_dir):
    """MARK a thousand positions back, seen and no longer seen, by rows of a prompt and by decoded tokens whose window is
    cut over several CTAs, beside other sequences."""
    config, tensors = standing_out(1100, dim=40, vdim=56)
    ids = [token if token != MARK else MARK + 1 for token in case.tokens(config, 1230, seed=4)]
    ids[70] = MARK
    want = case.truth(config, tensors, ids)[0]
    blind = case.truth(config, tensors, [8 if token == MARK else token for token in ids])[0]
    assert case.error(blind[1000:1169], want[1000:1169]) > 5 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype, slots=3, capacity=1264, max_rows=1264, max_wanted=1264) as ex:
        assert case.error(run_cut(ex, ids, [1230]), want) < case.TOLERANCE[dtype]
        slots = [ex.open() for _ in range(3)]
        starts = [1160, 300, 1120]                               # the first leaves MARK behind while it decodes
        for slot, start in zip(slots, starts):
            ex.run([Portion(slot, ids[:start])])
        for turn in range(25):
            got = ex.run([Portion(slot, [ids[start + turn]], [0]) for slot, start in zip(slots, starts)])
            assert case.error(got, want[[start + turn for start in starts]]) < case.TOLERANCE[dtype], turn


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_rest_on_the_null_key(dtype, plan_dir):
    """Heads of which one scores high, one near 0 and one far below: without the null key, or with one of another score,
    the first positions' outputs (each head's share of the whole) would differ."""
    config = case.model(40, 61, [case.layer(3, 1, 16, 12, 4, 20, scale=0.6)])
    tensors = case.weights(config, seed=8)
    tensors["embed"][:, 1] = 2.0
    tensors["l0.mix.k"][15, 1] = 3.0
    for head, size in enumerate((2.0, 0.0, -4.0)):
        tensors["l0.mix.q"][16 * head + 15, 1] = size
    tensors = bf16(tensors)
    ids = case.tokens(config, 40)
    want = case.truth(config, tensors, ids)[0]
    original = oracle.softmax_with_null
    for wrong in (lambda score, seen: torch.softmax(score.masked_fill(~seen, float("-inf")), -1),
                  lambda score, seen: original(score - 1.0, seen)):
        oracle.softmax_with_null = wrong
        try:
            other = case.truth(config, tensors, ids)[0]
        finally:
            oracle.softmax_with_null = original
        assert case.error(other[:4], want[:4]) > 3 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([40], [1], [2], [1, 39], [3, 1]):
            got = run_cut(ex, ids, cuts)
            assert case.error(got, want) < case.TOLERANCE[dtype] and case.error(got[:2], want[:2]) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
def test_scores_far_from_zero(dtype, plan_dir):
    """Scores in the hundreds, of both signs: a maximum above the null key's score and one far below it."""
    for sign in (1.0, -1.0):
        config = case.model(48, 61, [case.layer(4, 2, 16, 16, 4, 90, scale=sign * 20.0)])
        tensors = case.weights(config, seed=9)
        tensors["embed"][:, 1] = 3.0
        for part in ("q", "k"):
            tensors[f"l0.mix.{part}"][15::16, 1] = 2.0           # q . k > 0 throughout
        tensors = bf16(tensors)
        ids = case.tokens(config, 100)
        want = case.truth(config, tensors, ids)[0]
        assert torch.isfinite(want).all()
        with executor(config, tensors, plan_dir, dtype) as ex:
            for cuts in ([100], [60, 1]):
                got = run_cut(ex, ids, cuts)
                assert torch.isfinite(got).all()
                if sign < 0:
                    assert case.error(got, want) < case.TOLERANCE[dtype], cuts
                elif dtype == "f32":                             # (in bf16 rounding decides which of many keys scores highest)
                    assert case.error(got, want) < 30 * case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_over_all_heads_together(dtype, plan_dir):
    """Heads of very unequal size: a norm per head would bring them to the same size."""
    config = case.model(48, 61, [case.layer(6, 3, 16, 8, 8, 30, scale=0.7)])
    tensors = case.weights(config, seed=12)
    for head in range(6):
        tensors["l0.mix.q"][16 * head:16 * head + 16] *= 2.0 ** (head - 3)
    for head in range(3):
        tensors["l0.mix.k"][16 * head:16 * head + 16] *= 3.0 ** (1 - head)
    tensors = bf16(tensors)
    ids = case.tokens(config, 70)
    want = case.truth(config, tensors, ids)[0]
    original = oracle.rms_norm
    oracle.rms_norm = lambda x, w, eps: (original(x.reshape(len(x), -1, 16), w.reshape(-1, 16), eps).reshape(x.shape) if w.numel() == 96 or
                                         (w.numel() == 48 and torch.equal(w.float(), tensors["l0.mix.k.norm"])) else original(x, w, eps))
    try:
        other = case.truth(config, tensors, ids)[0]
    finally:
        oracle.rms_norm = original
    assert case.error(other, want) > 3 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([70], [33, 1], [2]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_positions_turn_by_their_own_scaled_angle(dtype, plan_dir):
    """A rotation over whole heads, thousands of positions from the start: angles and distances stay exact."""
    config = case.model(24, 40, [case.layer(2, 1, 16, 12, 16, 50, base=300.0, factor=2.0), case.layer(2, 2, 8, 8, 8, 30, base=90.0, factor=1.25)])
    tensors, ids = case.weights(config), case.tokens(config, 2000)
    want = case.truth(config, tensors, ids)[0]
    unscaled = copy.deepcopy(config)
    unscaled["layers"][0]["mixer"]["rot"]["scaling"]["factor"] = 1.0
    assert case.error(case.truth(unscaled, tensors, ids[:60])[0], want[:60]) > 3 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype, slots=1, capacity=2000, max_rows=1000) as ex:
        slot = ex.open()
        out = [ex.run([Portion(slot, ids[at:at + 650], [649])]) for at in (0, 650, 1300)]
        for at in range(1950, 2000):
            out.append(ex.run([Portion(slot, [ids[at]], [0])]))
    assert case.error(torch.cat(out), want[[649, 1299, 1949] + list(range(1950, 2000))]) < 2 * case.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_scores_weigh_what_the_experts_read(dtype, plan_dir):
    """A score beside an expert's output instead of its input, or scores that are made to sum to one, would show (the
    layer's norm hides their common size, not their ratios)."""
    config = case.model(64, 90, [case.layer(2, 1, 16, 16, 8, 20, case.moe(6, 3, 32))])
    tensors, ids = case.weights_for(config, dtype, seed=2), case.tokens(config, 75)
    tensors["l0.mlp.router"] *= 2.0
    tensors["embed"][:, 20], tensors["l0.norm1"][20], tensors["l0.mlp.router"][:, 20] = 2.5, 0.0, -1.0     # scores far apart
    want = case.truth(config, tensors, ids)[0]
    original = oracle.expert_mixture

    def on_output(x, spec, w):
        indices, scores = oracle.route(x, w("router"), spec["router"]["top"])
        rows = [sum(s * (oracle.squared_relu(x[t] @ w(f"e{e}.up").T) @ w(f"e{e}.down").T) for e, s in zip(indices[t].tolist(), scores[t]))
                for t in range(x.shape[0])]
        return torch.stack(rows)

    oracle.expert_mixture = on_output
    try:
        assert case.error(case.truth(config, tensors, ids)[0], want) > 3 * case.TOLERANCE[dtype]
    finally:
        oracle.expert_mixture = original
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([75], [63, 1], [64, 2], [65, 3]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts, top, favourite", [(24, 1, True), (24, 2, True), (24, 1, False), (200, 5, False), (3, 3, False)])
def test_routing_tables(experts, top, favourite, dtype, plan_dir):
    """Steps of 1 to 700 rows, around the size at which routing changes its form and at which tiles grow; all rows on the
    same expert (its tiles then outnumber those of an even spread), most experts without a row, every expert in use."""
    config = case.model(212, 130, [case.layer(2, 1, 16, 16, 8, 10, case.moe(experts, top, 40))])
    tensors = case.weights_for(config, dtype, seed=7)
    if favourite:                                                # one expert ahead of all others for every token
        tensors["embed"][:, experts + 1] = 4.0
        tensors["l0.norm1"][experts + 1] = 0.0
        tensors["l0.mlp.router"][:, experts + 1] = 0.0
        tensors["l0.mlp.router"][11, experts + 1] = 8.0
    ids = case.tokens(config, 700)
    want = case.truth(config, tensors, ids)[0]
    with executor(config, tensors, plan_dir, dtype, slots=1, capacity=704, max_rows=704, max_wanted=704) as ex:
        for cuts in ([700], [63, 64, 65, 128, 129, 251], [1, 2, 7, 33, 300, 357], [690, 1]):
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
