"""Faults that random weights would hide in a Benarax-shaped model: a far key, a rotation of the wrong pairs or of the wrong
length, a history lost or one token off, a state forgotten, a group's norm taken over all columns, another layer's part of
the second embedding. The weights are made so that each shows; wrong variants run in the plain forward only."""
import copy
import math

import pytest
import torch

import benarax_case as case
from oracle import benarax_oracle as oracle
from test_gpu_ragged import DTYPES, executor, run_cut
from tilemega_b200.serving.ragged import Portion

pytestmark = pytest.mark.gpu
MARK = 7          # the token that stands out


def bf16(tensors):
    return {name: tensor.to(torch.bfloat16).float() for name, tensor in tensors.items()}


def altered(name, wrong, config, tensors, ids):
    """The plain forward's logits with one of its functions replaced."""
    original = getattr(oracle, name)
    setattr(oracle, name, wrong(original))
    try:
        return case.truth(config, tensors, ids)[0]
    finally:
        setattr(oracle, name, original)


def marked(config, length, places, seed):
    ids = [token if token != MARK else MARK + 1 for token in case.tokens(config, length, seed=seed)]
    for place in places:
        ids[place] = MARK
    return ids


def without_mark(ids):
    return [8 if token == MARK else token for token in ids]


def quiet(config, tensors):
    """Only the first layer's mixer matters: no convolution, and side inputs that add little."""
    for name, tensor in tensors.items():
        if name.endswith("canon1"):
            tensor.zero_()
        elif name.endswith("side.norm"):
            tensor *= 0.05


def standing_out(**sizes):
    """One latent layer in which every query points along one (unrotated) direction and only MARK's key lies along it: MARK takes
    nearly all of the weight wherever it is behind."""
    sizes = dict(heads=4, dim=24, rot=8, vdim=18, rank=20, q_rank=16, scale=0.5) | sizes
    config = case.model(40, 61, [case.latent(**sizes)], side=4, embed_scale=1.0)
    tensors, dim, rot = case.weights(config, seed=3), sizes["dim"], sizes["rot"]
    tensors["embed"][:, 0] = 0.0
    tensors["embed"][:, 1] = 1.0                                 # every token
    tensors["embed"][MARK, 2:] *= 0.1
    tensors["embed"][MARK, 0] = 4.0                              # alone in column 0
    quiet(config, tensors)
    tensors["l0.mix.dq"].mul_(0.05)
    tensors["l0.mix.dq"][0] = 0.0
    tensors["l0.mix.dq"][0, 1] = 3.0
    tensors["l0.mix.uq"].mul_(0.05)
    tensors["l0.mix.uq"].view(sizes["heads"], dim + rot, -1)[:, dim - 1, 0] = 2.0
    tensors["l0.mix.dkv"][0] = 0.0
    tensors["l0.mix.dkv"][0, 0] = 4.0                            # MARK's latent row alone has an entry 0
    tensors["l0.mix.uk"][dim - 1::dim] = 0.0
    tensors["l0.mix.uk"][dim - 1::dim, 0] = 3.0
    tensors["l0.mix.uv"][:, 0] = torch.linspace(-1, 1, len(tensors["l0.mix.uv"]))
    return config, bf16(tensors)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank", [20, 90, 500, 570, 650])       # (long portions expand wide rows only; the last is wider than the tiles)
def test_a_key_at_block_borders(rank, dtype, plan_dir):
    """MARK as the first token, the last of a block, the first of the next: seen at once and from then on."""
    config, tensors = standing_out(rank=rank)
    with executor(config, tensors, plan_dir, dtype, capacity=256) as ex:
        for place in (0, 1, 15, 16, 63, 64, 65):
            ids = marked(config, place + 80, [place], seed=place)
            want = case.truth(config, tensors, ids)[0]
            blind = case.truth(config, tensors, without_mark(ids))[0]
            assert case.error(blind[place + 1:], want[place + 1:]) > 5 * case.TOLERANCE[dtype]
            for cuts in ([len(ids)], [place + 1, 1], [place + 17, 2], [5, 2, 33, 1]):
                assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], (place, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [dict(dim=40, vdim=56, rank=30), dict(dim=16, vdim=16, rank=200, heads=40, neighbours=False),
                                   dict(dim=16, vdim=24, rot=64, rank=450, heads=70), dict(dim=64, rot=32, vdim=32, rank=600)])
def test_a_far_key_among_a_thousand(sizes, dtype, plan_dir):
    """MARK a thousand positions back, by rows of a prompt and by decoded tokens whose keys are cut over several CTAs, beside
    other sequences, one of which has not seen it."""
    config, tensors = standing_out(**sizes)
    ids = marked(config, 1230, [70], seed=4)
    want = case.truth(config, tensors, ids)[0]
    blind = case.truth(config, tensors, without_mark(ids))[0]
    assert case.error(blind[1000:], want[1000:]) > 5 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype, slots=3, capacity=1264, max_rows=1264, max_wanted=1264) as ex:
        for cuts in ([1230], [1100, 130], [600, 500, 2, 3, 125]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts
        slots = [ex.open() for _ in range(3)]
        starts = [1160, 45, 1120]
        for slot, start in zip(slots, starts):
            ex.run([Portion(slot, ids[:start])])
        for turn in range(30):
            got = ex.run([Portion(slot, [ids[start + turn]], [0]) for slot, start in zip(slots, starts)])
            expected = want[[start + turn for start in starts]]
            assert (got - expected).pow(2).mean(-1).sqrt().max() < case.TOLERANCE[dtype] * want.pow(2).mean().sqrt(), turn


def turning(neighbours, scaling=None, base=30.0, **sizes):
    """One latent layer whose scores come from the rotated parts alone: MARK is found at certain distances only."""
    sizes = dict(heads=3, dim=4, rot=16, vdim=20, rank=24, q_rank=20, scale=1.0) | sizes
    config = case.model(40, 61, [case.latent(**sizes, neighbours=neighbours, scaling=scaling, base=base)], side=4, embed_scale=1.0)
    tensors, dim, rot = case.weights(config, seed=5), sizes["dim"], sizes["rot"]
    quiet(config, tensors)
    tensors["embed"][:, 1] = 1.0
    tensors["l0.mix.dq"].mul_(0.02)
    tensors["l0.mix.dq"][0, 1] = 2.0                             # the same query for every token
    tensors["l0.mix.uq"].mul_(0.02)
    heads = tensors["l0.mix.uq"].view(sizes["heads"], dim + rot, -1)
    generator = torch.Generator().manual_seed(2)
    heads[:, dim:, 0] = 0.4 * torch.randn((sizes["heads"], rot), generator=generator)
    tensors["l0.mix.uk"].mul_(0.02)
    tail = tensors["l0.mix.dkv"][sizes["rank"]:]
    tail.mul_(0.1)
    tail[:, 1] = torch.randn(rot, generator=generator)           # the same rotated key for every token
    return config, bf16(tensors)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("neighbours, scaling", [(True, None), (False, None), (True, case.stretch(4.0, 256, 6.0, 1.0)), (True, case.stretch(2.0, 40, 1.5, 1.0)),
                                                 (False, case.stretch(16.0, 2000, 32.0, 0.5))])
def test_rotations(neighbours, scaling, dtype, plan_dir):
    """The other layout, an unscaled or fully scaled rotation, or its size left out would show; near the start and hundreds of
    positions from it."""
    config, tensors = turning(neighbours, scaling)
    ids = case.tokens(config, 400)
    want = case.truth(config, tensors, ids)[0]
    wrong = [("rotate", lambda f: lambda x, p, rot, n: f(x, p, rot, not n)), ("rotate", lambda f: lambda x, p, rot, n: f(x, p + 0 * p, rot | {"base": 31.0}, n))]
    if scaling:
        wrong += [("frequencies", lambda f: lambda rot: (f({**rot, "scaling": None})[0], f(rot)[1])), ("frequencies", lambda f: lambda rot: (f(rot)[0], 1.0)),
                  ("frequencies", lambda f: lambda rot: ([t / rot["scaling"]["factor"] for t in f({**rot, "scaling": None})[0]], f(rot)[1]))]
    for name, variant in wrong:
        assert case.error(altered(name, variant, config, tensors, ids), want) > case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype, slots=2) as ex:
        for cuts in ([400], [1], [33, 2, 1], [300, 3]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_positions_keep_their_angles(dtype, plan_dir):
    config, tensors = turning(True, case.stretch(2.0, 500, 8.0, 1.0), base=10000.0)
    ids = case.tokens(config, 2000)
    want = case.truth(config, tensors, ids)[0]
    with executor(config, tensors, plan_dir, dtype, slots=1, capacity=2000, max_rows=1000) as ex:
        slot = ex.open()
        out = [ex.run([Portion(slot, ids[at:at + 650], [649])]) for at in (0, 650, 1300)]
        for at in range(1950, 2000):
            out.append(ex.run([Portion(slot, [ids[at]], [0])]))
    assert case.error(torch.cat(out), want[[649, 1299, 1949] + list(range(1950, 2000))]) < case.TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_scores_far_from_zero(dtype, plan_dir):
    """Scores of hundreds, above zero and below it."""
    for scale in (25.0, -25.0):
        config, tensors = standing_out(scale=scale)
        ids = marked(config, 100, [3, 40], seed=6)
        want = case.truth(config, tensors, ids)[0]
        assert torch.isfinite(want).all()
        with executor(config, tensors, plan_dir, dtype) as ex:
            for cuts in ([100], [60, 1]):
                got = run_cut(ex, ids, cuts)
                assert torch.isfinite(got).all() and case.error(got, want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 8, 9, 16])
@pytest.mark.parametrize("width, groups", [(48, 4), (50, 5)])
def test_short_convolutions(taps, width, groups, dtype, plan_dir):
    """Convolutions that outweigh the norm itself: taps in the other order, a history one token short, a feed-forward that reads
    them too would show. Portions shorter and longer than a convolution and than what one CTA walks; widths with and without the
    vectorised form."""
    config = case.model(width, 61, [case.latent(2, 8, 4, 12, 10, 9, case.moe(3, 1, 16)), case.delta(2, 16, 4, case.moe(2, 1, 24))], groups=groups, taps=taps, loop=(0, 2, 2), eps=1e-2)
    tensors = case.weights_for(config, dtype, seed=taps)
    for name, tensor in tensors.items():
        if name.endswith("canon1"):
            tensor *= 2.0
    tensors = bf16(tensors)
    ids = case.tokens(config, 330)
    want = case.truth(config, tensors, ids)[0]
    if taps > 1:
        def short(f):
            def convolve(h, kernel):
                kernel = kernel.clone()
                kernel[:, 0] = 0.0
                return f(h, kernel)
            return convolve
        for wrong in (lambda f: lambda h, kernel: f(h, kernel.flip(1)), short):
            assert case.error(altered("short_convolution", wrong, config, tensors, ids[:60]), want[:60]) > 2 * case.TOLERANCE[dtype]
    cases = ([330], [1], [2], [3, 1], [taps, 1], [max(1, taps - 1)], [taps + 1, 2], [17, 100, 1, 2, 5], [300, 2, 1])
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in cases:
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts
        # several sequences whose portions differ in length, in one step
        slots = [ex.open() for _ in range(4)]
        done = [0, 0, 0, 0]
        for sizes in ((1, 40, 2, taps), (90, 1, 7, 1), (2, 3, 1, 64), (1, 1, 1, 1)):
            got, at = ex.run([Portion(slot, ids[d:d + n], list(range(n))) for slot, d, n in zip(slots, done, sizes)]), 0
            for index, n in enumerate(sizes):
                difference = (got[at:at + n] - want[done[index]:done[index] + n]).pow(2).mean(-1).sqrt().max()
                assert difference < case.TOLERANCE[dtype] * want.pow(2).mean().sqrt(), (sizes, index)
                at, done[index] = at + n, done[index] + n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim, heads", [(20, 3), (64, 2), (96, 2), (128, 1), (192, 1), (208, 2)])
def test_states_that_remember(dim, heads, dtype, plan_dir):
    """Decays near one and removals near zero: what MARK wrote is read hundreds of tokens later. Removal of another key's share,
    a removal that reads the state after its decay, or a write of the unit key would show."""
    config = case.model(48, 61, [case.delta(heads, dim, 6)], side=4, embed_scale=1.0, taps=2)
    tensors = case.weights(config, seed=dim)
    quiet(config, tensors)
    tensors["embed"][:, 0] = 0.0
    tensors["embed"][:, 1] = 1.0
    tensors["embed"][MARK] *= 0.1
    tensors["embed"][MARK, 0] = 6.0
    for part in ("r", "k", "v"):
        tensors[f"l0.mix.{part}"].mul_(0.1)
    tensors["l0.mix.k"][::dim, 0] = 3.0                          # MARK writes one key channel, every token reads it
    tensors["l0.mix.r"][::dim, 1] = 3.0
    tensors["l0.mix.v"][:, 0] = torch.linspace(-1, 1, heads * dim)
    tensors["l0.mix.w0"].fill_(-9.0)
    tensors["l0.mix.a.b"].fill_(-9.0)
    slow = bf16(tensors)
    ids = marked(config, 600, [20], seed=5)
    want = case.truth(config, slow, ids)[0]
    assert case.error(case.truth(config, slow, without_mark(ids))[0][400:], want[400:]) > 5 * case.TOLERANCE[dtype]
    with executor(config, slow, plan_dir, dtype, capacity=608, max_rows=608, max_wanted=608) as ex:
        for cuts in ([600], [21, 1], [300, 2, 33, 1], [7, 64, 9]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts
    # decays and removals of all sizes, keys far from unit length that come again and again
    tensors = case.weights(config, seed=dim + 1)
    for part in ("w0", "a.b"):
        tensors[f"l0.mix.{part}"].mul_(3.0)
    tensors["l0.mix.k"].mul_(2.0)
    tensors["embed"][:, :8] = tensors["embed"][0, :8]            # much of every key is the same
    tensors = bf16(tensors)
    ids = case.tokens(config, 200)
    want = case.truth(config, tensors, ids)[0]

    def after_decay(f):
        def recurrence(r, k, v, w, a):
            state, out = torch.zeros(r.shape[1], v.shape[1], dtype=r.dtype), torch.empty_like(v)
            for t in range(len(r)):
                u = k[t] / torch.sqrt((k[t] * k[t]).sum() + 1e-6)
                state = w[t][:, None] * state
                state = state - torch.outer(a[t] * u, u @ state) + torch.outer(k[t], v[t])
                out[t] = r[t] @ state
            return out
        return recurrence

    # decays as steep as they get, and removals of everything
    steep = bf16(tensors | {"l0.mix.w0": torch.full_like(tensors["l0.mix.w0"], 9.0), "l0.mix.a.b": torch.full_like(tensors["l0.mix.a.b"], 9.0)})
    expected = case.truth(config, steep, ids)[0]
    with executor(config, steep, plan_dir, dtype) as ex:
        for cuts in ([200], [1], [13, 21, 2]):
            assert case.error(run_cut(ex, ids, cuts), expected) < case.TOLERANCE[dtype], cuts

    if dtype == "f32":
        unit = lambda k: k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        for name, wrong in (("delta_recurrence", after_decay), ("delta_recurrence", lambda f: lambda r, k, v, w, a: f(r, unit(k), v, w, a)),
                            ("delta_recurrence", lambda f: lambda r, k, v, w, a: f(r, k, v, w, 0 * a)),
                            ("decay_of", lambda f: lambda z: torch.sigmoid(z))):
            assert case.error(altered(name, wrong, config, tensors, ids), want) > 20 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([200], [1], [8, 9, 1, 7], [100, 2]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, groups", [(48, 1), (48, 2), (48, 16), (1024, 4), (1024, 8), (50, 10), (49, 7), (3072, 3), (4104, 6)])
def test_groups_of_columns(width, groups, dtype, plan_dir):
    """Groups of very unequal size: one norm over all columns, or other groups, would show. Widths of each form of the kernel."""
    config = case.model(width, 61, [case.latent(2, 8, 4, 12, 10, 9), case.delta(2, 16, 4)], groups=groups, taps=2)
    tensors = case.weights(config, seed=groups)
    for group, part in enumerate(tensors["embed"].chunk(groups, dim=1)):
        part *= 3.0 ** (group % 4 - 1)
    tensors = bf16(tensors)
    ids = case.tokens(config, 60)
    want = case.truth(config, tensors, ids)[0]
    if groups > 1:
        assert case.error(case.truth(config | {"norm": {"eps": 1e-5, "groups": 1}}, tensors, ids)[0], want) > 2 * case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([60], [1], [2], [33, 1]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("side", [1, 6, 40, 130])
def test_side_inputs(side, dtype, plan_dir):
    """Side inputs that outweigh the sublayers: another layer's part, a part per pass, a plain sigmoid-free gate or a gate of the
    normed stream would show."""
    config = case.model(48, 61, [case.latent(2, 8, 4, 12, 10, 9), case.delta(2, 16, 4), case.delta(2, 16, 4)], side=side, groups=2, loop=(0, 2, 2))
    tensors = case.weights(config, seed=side)
    for name, tensor in tensors.items():
        if name.endswith("side.norm"):
            tensor *= 3.0
        elif name.endswith("side.gate") and side > 1:
            tensor *= 2.0
        elif name.endswith("side.gate"):                         # (the sign of a single product hangs on rounding)
            tensor.abs_()
    if side == 1:
        tensors["embed"].abs_()
        tensors["embed"] += 2.0
        tensors["side.embed"].abs_()
        tensors["side.embed"] += 1.0
    tensors = bf16(tensors)
    ids = case.tokens(config, 80)
    want = case.truth(config, tensors, ids)[0]
    if side > 1:
        moved = dict(tensors) | {"side.embed": tensors["side.embed"].roll(side, dims=1)}
        assert case.error(case.truth(config, moved, ids)[0], want) > 2 * case.TOLERANCE[dtype]
        for wrong in (lambda f: lambda z: torch.relu(z), lambda f: lambda z: z):
            assert case.error(altered("gelu_tanh", wrong, config, tensors, ids), want) > case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([80], [1], [2], [33, 1]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("factors", [dict(residual_mult=0.25), dict(embed_scale=7.0), dict(logit_scale=3.0), dict(residual_mult=1.0, embed_scale=0.3, logit_scale=1.0)])
def test_factors(factors, dtype, plan_dir):
    config = case.model(48, 61, [case.latent(2, 8, 4, 12, 10, 9, case.moe(3, 1, 16)), case.delta(2, 16, 4)], **factors)
    tensors, ids = case.weights_for(config, dtype), case.tokens(config, 70)
    want = case.truth(config, tensors, ids)[0]
    with executor(config, tensors, plan_dir, dtype) as ex:
        for cuts in ([70], [30, 1]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts, top", [(24, 1), (24, 5), (200, 5), (12, 12), (300, 6), (40, 32)])
def test_routing(experts, top, dtype, plan_dir):
    """Steps of 1 to 700 rows, around the sizes at which routing changes its form and at which tiles grow."""
    if dtype == "bf16" and experts == 300:
        pytest.skip("three hundred levels lie too close together for 16 bits")
    config = case.model(340, 130, [case.latent(2, 16, 4, 16, 8, 8, case.moe(experts, top, 40))])
    tensors, ids = case.weights_for(config, dtype, seed=7), case.tokens(config, 700)
    want = case.truth(config, tensors, ids)[0]
    with executor(config, tensors, plan_dir, dtype, slots=1, capacity=704, max_rows=704, max_wanted=704) as ex:
        for cuts in ([700], [63, 64, 65, 128, 129, 251], [1, 2, 7, 33, 300, 357], [690, 1]):
            assert case.error(run_cut(ex, ids, cuts), want) < case.TOLERANCE[dtype], cuts


def test_logits_of_hundreds_still_rank_experts(plan_dir):
    """One expert's logit stands so far above the others that their shares of a softmax over all of them vanish: the second
    choice is still the second largest."""
    config = case.model(64, 90, [case.latent(2, 16, 4, 16, 24, 8, case.moe(9, 3, 32))])
    tensors, ids = case.weights(config, seed=2), case.tokens(config, 75)
    tensors["embed"][:, 1] = 2.0
    tensors["l0.mlp.router"].mul_(60.0)
    tensors["l0.mlp.router"][8, 1] = 400.0                       # always first, and far off
    tensors = bf16(tensors)
    want, seen = case.truth(config, tensors, ids)[0], []
    altered("route", lambda f: lambda z, top: (seen.append(z), f(z, top))[1], config, tensors, ids)
    assert min(float(z.max() - z.sort().values[-2]) for z in seen) > 110
    with executor(config, tensors, plan_dir, "f32") as ex:
        slot = ex.open()
        ex.run([Portion(slot, ids[:5])])
        for wide in (False, True):
            got = run_cut(ex, ids, [75] if wide else [3])
            assert case.error(got, want) < case.TOLERANCE["f32"]
        choices = torch.stack([z.topk(3).indices for z in seen])
        assert len(choices[:, 1].unique()) > 4                   # (and it is not always the same)


@pytest.mark.parametrize("dtype", DTYPES)
def test_limits_of_experts(dtype, plan_dir):
    """Activations well beyond the limit: one left out, or half as high, would show."""
    config = case.model(64, 90, [case.latent(2, 16, 4, 16, 24, 8, case.moe(4, 2, 32, limit=0.9))])
    tensors, ids = case.weights_for(config, dtype, seed=2), case.tokens(config, 75)
    for name, tensor in tensors.items():
        if name.endswith((".gate", ".up")) and "side" not in name:
            tensor *= 3.0
    tensors = bf16(tensors)
    want = case.truth(config, tensors, ids)[0]
    for limit in (0.45, 50.0):
        other = copy.deepcopy(config)
        other["layers"][0]["mlp"]["expert"]["limit"] = limit
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
    scale = math.sqrt(torch.cat(wanted).pow(2).mean())
    with executor(config, tensors, plan_dir, "bf16", slots=70, capacity=32, max_rows=1120) as ex:
        slots = [ex.open() for _ in ids]
        ex.run([Portion(slot, sequence[:16]) for slot, sequence in zip(slots, ids)])
        for turn, count in enumerate((70, 64, 65, 33, 16, 3, 1, 70)):
            done = [16 + sum(1 for c in (70, 64, 65, 33, 16, 3, 1)[:turn] if index < c) for index in range(70)]
            got = ex.run([Portion(slots[index], [ids[index][done[index]]], [0]) for index in range(count)])
            want = torch.stack([wanted[index][done[index]] for index in range(count)])
            assert (got - want).pow(2).mean(-1).sqrt().max() < case.TOLERANCE["bf16"] * scale, count
