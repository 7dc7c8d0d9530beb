"""Benarax on the GPU against the plain forward of oracle/benarax_oracle.py: every case of benarax_case.py in fp32 and
bf16, however the tokens are cut into steps, whatever shares the batch, on used pages and slots."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import benarax_case as case
from test_gpu_ragged import DTYPES, executor, run_cut
from tilemega_b200.planbuild import emit_plan
from tilemega_b200.serving.continuous import ContinuousEngine, Request
from tilemega_b200.serving.ragged import Portion
from tilemega_b200.serving.weights import TensorCheckpoint

pytestmark = pytest.mark.gpu
STATES = ("kv_pool", "delta", "history")


@pytest.mark.parametrize("name, dtype", case.RUNS)
def test_prompts_cut_anywhere(name, dtype, plan_dir):
    """One step, token by token, portions down to two tokens, portions that end at and beside block edges and shorter and
    longer than a convolution: all the same logits, those of the plain forward; and the residual stream after every layer run."""
    config = case.CASES[name]
    tensors, ids = case.weights_for(config, dtype), case.tokens(config, 150)
    want, kept = case.truth(config, tensors, ids)
    tolerance = case.TOLERANCE[dtype]
    with executor(config, tensors, plan_dir, dtype, write_residuals=True) as ex:
        whole = run_cut(ex, ids, [len(ids)])
        for got, expected in zip(ex.residuals(len(ids)), kept):
            assert case.error(got, expected) < tolerance
        assert case.error(whole, want) < tolerance
        for cuts in ([1], [2], [3, 1, 2, 64, 1, 17], [16, 48, 1, 1, 63], [65, 2, 1], [100, 1], [31, 33, 5]):
            assert case.error(run_cut(ex, ids, cuts), want) < tolerance, cuts
    with executor(config, tensors, plan_dir, dtype) as ex:       # (plans without residuals record and replay decode steps)
        assert case.error(run_cut(ex, ids, [40, 1]), want) < tolerance


@pytest.mark.parametrize("name, dtype", case.RUNS)
def test_mixed_batches_on_used_pages_and_slots(name, dtype, plan_dir):
    """Up to four sequences at once, portions beside single tokens, some left out of a step; more sequences than slots
    over a pool that only just holds four. Pools, states and histories start as garbage."""
    config = case.CASES[name]
    tensors = case.weights_for(config, dtype)
    lengths = [70, 1, 33, 120, 2, 49, 18, 90]
    prompts = [case.tokens(config, length, seed=10 + index) for index, length in enumerate(lengths)]
    wanted = [case.truth(config, tensors, ids)[0] for ids in prompts]
    scale = torch.cat(wanted).pow(2).mean().sqrt()
    generator = torch.Generator().manual_seed(9)
    pick = lambda high: int(torch.randint(0, high, (1,), generator=generator))
    with executor(config, tensors, plan_dir, dtype, capacity=128, num_blocks=22) as ex:
        for key, tensor in ex.state.items():
            if key.startswith(STATES):
                tensor.fill_(3.0)
        waiting, live, got = list(range(len(prompts))), {}, {index: [] for index in range(len(prompts))}
        while waiting or live:
            while waiting and len(live) < 4:
                live[waiting.pop(0)] = [ex.open(), 0]
            portions, owners = [], []
            for index, (slot, done) in live.items():
                if len(live) > 1 and pick(5) == 0:
                    continue
                size = min([1, 1, 2, 3, 16, 29, 64][pick(7)], lengths[index] - done)
                portions.append(Portion(slot, prompts[index][done:done + size], list(range(size))))
                owners.append(index)
            if not portions:
                continue
            logits, at = ex.run(portions), 0
            for index, portion in zip(owners, portions):
                got[index].append(logits[at:at + len(portion.tokens)])
                at += len(portion.tokens)
                live[index][1] += len(portion.tokens)
                if live[index][1] == lengths[index]:
                    ex.close_sequence(live.pop(index)[0])
        for index, expected in enumerate(wanted):
            assert (torch.cat(got[index]) - expected).pow(2).mean(-1).sqrt().max() < case.TOLERANCE[dtype] * scale, index
        assert len(ex.sequences.pool.free) == 21 and len(ex.sequences.free) == 4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "crowd"])
def test_long_decoding(name, dtype, plan_dir):
    """Hundreds of decoded tokens over many pages: ahead on the device and step by step."""
    config = case.CASES[name]
    tensors, prompt = case.weights_for(config, dtype), case.tokens(config, 9)
    with executor(config, tensors, plan_dir, dtype) as ex:
        slot, steps = ex.open(), 330
        first = ex.step([Portion(slot, prompt, [len(prompt) - 1])])[0][0]
        ahead = ex.decode_ahead({slot: first}, steps)[slot]
        ex.close_sequence(slot)
        ids = prompt + [first] + ahead
        want = case.truth(config, tensors, ids[:-1])[0]
        assert case.error(run_cut(ex, ids[:-1], [len(prompt), 1]), want) < case.TOLERANCE[dtype]
        chosen = want[len(prompt) - 1:].gather(1, torch.tensor(ids[len(prompt):])[:, None])[:, 0]
        slack = 2 * case.TOLERANCE[dtype] * want.pow(2).mean().sqrt() * 4
        assert (want[len(prompt) - 1:].max(-1).values - chosen <= slack).all()


@pytest.mark.parametrize("decode_chunk", [1, 5])
def test_greedy_generation_through_the_continuous_engine(decode_chunk, plan_dir):
    """More requests than slots, prompts longer than a step; every request generates the plain forward's greedy tokens."""
    config = case.CASES["odd"]
    tensors = case.weights(config)
    shapes = [(5, 12), (40, 3), (1, 20), (23, 1), (64, 9)]
    requests = [Request(index, case.tokens(config, length, seed=30 + index), new) for index, (length, new) in enumerate(shapes)]
    expected = {}
    for request in requests:
        ids = list(request.prompt)
        for _ in range(request.max_new_tokens):
            ids.append(int(case.truth(config, tensors, ids)[0][-1].argmax()))
        expected[request.id] = ids[len(request.prompt):]
    so = emit_plan(config, plan_dir, phase="ragged", slots=2, capacity=96, num_blocks=10, max_rows=17, dtype="f32")
    with ContinuousEngine(TensorCheckpoint(tensors), config, so, 2, decode_chunk=decode_chunk) as engine:
        for request in requests:
            engine.submit(request)
        finished = engine.run_until_done()
        assert {request.id: request.generated for request in finished} == expected
        assert len(engine.scheduler.pool.free) == 9 and len(engine.ragged.sequences.free) == 2


@pytest.mark.parametrize("experts, top", [(16, 3), (128, 8)])
def test_products_at_model_widths(experts, top, plan_dir):
    """Widths at which every tile width and K split is in use, latent rows that long portions expand and short ones do not: a
    prompt in portions of 300, 100, 50, 20, 3 and single tokens, alone and beside another sequence."""
    config = case.model(2048, 500, [case.latent(16, 128, 64, 96, 512, 768, case.moe(experts, top, 512)), case.delta(16, 128, 96, case.moe(experts, top, 512)),
                                    case.latent(32, 64, 32, 128, 224, 512, neighbours=False), case.delta(8, 64, 32)], groups=8, taps=4, side=256)
    tensors, ids = case.weights(config, coded=True), case.tokens(config, 480)
    want = case.benarax_oracle.forward(config, tensors, ids, torch.float32)[0]
    with executor(config, tensors, plan_dir, "bf16", slots=2, capacity=512) as ex:
        assert case.error(run_cut(ex, ids, [300, 100, 50, 20, 3, 1]), want) < case.TOLERANCE["bf16"]
        other = ex.open()
        ex.run([Portion(other, ids[:200])])
        slot = ex.open()
        ex.run([Portion(slot, ids[:460])])
        for at in range(460, 470):
            pair = ex.run([Portion(other, [ids[at - 260]], [0]), Portion(slot, [ids[at]], [0])])
            assert case.error(pair, want[[at - 260, at]]) < case.TOLERANCE["bf16"]
        pair = ex.run([Portion(other, ids[210:400], [0, 120, 189]), Portion(slot, [ids[470]], [0])])     # a long portion beside a decoded token
        assert case.error(pair, want[[210, 330, 399, 470]]) < case.TOLERANCE["bf16"]


def write_model(folder, config, tensors):
    """A model folder; sizes that only the tensors' shapes tell are not in its config.json."""
    from safetensors.torch import save_file
    plain = json.loads(json.dumps(config))
    for layer in plain["layers"]:
        layer["mixer"].pop("decay_rank", None)
    (folder / "config.json").write_text(json.dumps(plain))
    save_file({name: tensor.to(torch.bfloat16).contiguous() for name, tensor in tensors.items()}, folder / "model.safetensors")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_replays_steps(dtype, tmp_path):
    """bin/trace_run: requests cut into steps, four live at once, ended and followed by others."""
    config = case.CASES["odd"]
    tensors = case.weights_for(config, "f32" if dtype == "float32" else "bf16")
    model = tmp_path / "model"
    model.mkdir()
    write_model(model, config, tensors)
    ids = {name: case.tokens(config, length, seed=length) for name, length in (("a", 70), ("b", 9), ("c", 33), ("d", 64), ("e", 20))}
    steps = [([("a", 0, 40, [0, 39]), ("b", 0, 5, [])], []), ([("b", 5, 9, [3, 0]), ("c", 0, 2, [1]), ("a", 40, 41, [0])], ["b"]),
             ([("d", 0, 64, [63, 62]), ("e", 0, 3, [2]), ("c", 2, 33, [30])], ["c"]), ([("a", 41, 70, [28])], ["a", "d"]), ([("e", 3, 20, [])], [])]
    lines, wanted = [], {}
    for number, (entries, end) in enumerate(steps):
        lines.append(json.dumps({"step": number, "entries": [{"id": name, "tokens": ids[name][lo:hi], "want": want} for name, lo, hi, want in entries],
                                 "end": end}))
        wanted[number] = [case.truth(config, tensors, ids[name])[0][lo + place] for name, lo, hi, want in entries for place in want]
    out = tmp_path / "out"
    out.mkdir()
    root = Path(__file__).resolve().parents[1]
    run = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(model), "--dtype", dtype, "--out", str(out),
                          "--max-tokens", "320"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [line for line in run.stdout.splitlines() if line.startswith("done")] == [f"done {number}" for number in range(len(steps))]
    for number, rows in wanted.items():
        path = out / f"{number}.f32"
        assert path.exists() == bool(rows)
        if rows:
            got = torch.frombuffer(bytearray(path.read_bytes()), dtype=torch.float32).reshape(len(rows), config["vocab"])
            assert case.error(got, torch.stack(rows)) < case.TOLERANCE["f32" if dtype == "float32" else "bf16"]


def test_generate_command_line(tmp_path, capsys):
    from tilemega_b200 import generate
    config = case.CASES["crowd"]
    tensors = case.weights(config)
    prompts = [case.tokens(config, length, seed=60 + length) for length in (7, 30, 2)]
    write_model(tmp_path, config, tensors)
    arguments = ["--model", str(tmp_path), "--dtype", "f32", "--new-tokens", "6", "--batch", "2", "--step-rows", "11"]
    for prompt in prompts:
        arguments += ["--prompt", " ".join(map(str, prompt))]
    assert generate.main(arguments) == 0
    printed = {line["request"]: line["generated"] for line in map(json.loads, capsys.readouterr().out.splitlines())}
    for number, prompt in enumerate(prompts):
        ids = list(prompt)
        for _ in range(6):
            ids.append(int(case.truth(config, tensors, ids)[0][-1].argmax()))
        assert printed[number] == ids[len(prompt):]
