"""Dozetar through the engine against the plain implementation, in 32-bit and in bfloat16, under every way of cutting
the work, at five small configurations that differ in every size and option (tests/dozetar_tools.py)."""
import pytest
import torch

import plain_dozetar as plain
from trace_tools import mixed_steps, portion_steps, tail_steps, whole_steps
from dozetar_tools import CONFIGS, make_tensors, plain_tensors, random_requests

pytestmark = pytest.mark.gpu

LENGTHS = {"A": [1, 5, 19, 20, 21, 41, 100, 130], "B": [2, 6, 7, 8, 15, 50, 64, 90], "C": [1, 99, 100, 101, 134, 260, 300, 201],
           "D": [1, 32, 33, 34, 67, 150, 9, 99], "E": [1, 49, 50, 51, 128, 129, 260, 77]}
FLOAT32_TOL = 2e-4
TOL = {}


@pytest.fixture(scope="module")
def models():
    out = {}
    for name, config in CONFIGS.items():
        for dtype in ("float32", "bfloat16"):
            tensors = make_tensors(config, seed=len(name) + ord(name), dtype=getattr(torch, dtype), decided=dtype == "bfloat16")
            requests = random_requests(config, LENGTHS[name], 11)
            reference = plain_tensors(tensors)
            want = {r: plain.forward(config, reference, t).float() for r, t in requests.items()}
            out[name, dtype] = (config, tensors, requests, want)
            # (a head's read-out that nearly vanishes before it is divided by its root mean square amplifies rounding: four times
            # what float32 does to the plain implementation itself comes on top)
            TOL[name, dtype] = FLOAT32_TOL + 4.0 * max((plain.forward(config, tensors, t) - want[r]).abs().max().item()
                                                       for r, t in requests.items()) if dtype == "float32" else None
            if dtype == "bfloat16":
                # the root mean square of a row's error, against three times what rounding the stored activations to
                # bfloat16 does to the plain implementation's own rows (a wrong or missing key, or a lost state, moves
                # a row by its whole spread, which is about one)
                plain.ROUND = torch.bfloat16
                moved = max((plain.forward(config, reference, t).float() - want[r]).square().mean(-1).sqrt().max().item()
                            for r, t in requests.items())
                plain.ROUND = None
                TOL[name, dtype] = -(3.0 * moved + 5e-3)
    return out


def engine_for(config, tensors, dtype, kv_tokens, page_size=16, max_requests=4, poison=True, **more):
    from damendaemon_b200.engine import Engine
    engine = Engine(config=config, tensors=tensors, dtype=dtype, kv_tokens=kv_tokens, page_size=page_size,
                    max_requests=max_requests, **more)
    if poison:
        for g in engine.cache.groups:
            g.arena.fill_(float("nan"))      # whatever was never written must never be read
        for state in engine.cache._all_states():
            state.fill_(float("nan") if state.is_floating_point() else 12345)   # a slot's states are zeroed when it is taken
    return engine


def replay(engine, builder):
    from damendaemon_b200.engine import StepEntry
    got = {}
    for s in builder.steps:
        entries = [StepEntry(e["id"], e["tokens"], e["want"]) for e in s["entries"]]
        if entries:
            logits = engine.step(entries).cpu()
            for (request, position), row in zip(builder.where[s["step"]], logits):
                got.setdefault(request, {})[position] = row
        for r in s["end"]:
            engine.finish(r)
        engine.cache.check()
    return got


def compare(got, want, tol, what):
    """tol > 0: the largest difference of a row; tol < 0: its root mean square, against -tol."""
    worst = 0.0
    for r, rows in got.items():
        for p in sorted(rows):
            assert torch.isfinite(rows[p]).all(), f"{what}: non-finite logits at request {r} position {p}"
            err = (rows[p] - want[r][p]).abs().max().item() if tol > 0 else (rows[p] - want[r][p]).square().mean().sqrt().item()
            worst = max(worst, err)
            assert err < abs(tol), f"{what}: request {r} position {p} differs by {err:.3e} (first wrong place)"
    for r in want:
        assert set(got[r]) == set(range(len(want[r]))), f"{what}: request {r} misses positions"
    return worst


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(models, name, dtype):
    config, tensors, requests, want = models[name, dtype]
    engine = engine_for(config, tensors, dtype, kv_tokens=320, page_size=16)
    compare(replay(engine, whole_steps(requests)), want, TOL[name, dtype], f"{name} {dtype} whole")
    assert engine.cache.used_tokens == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_then_token_by_token(models, name, dtype):
    """The last 45 tokens one by one: the windows pass over decoded tokens, and the memories with their maxima are carried from
    the prompt into single-token steps."""
    config, tensors, requests, want = models[name, dtype]
    engine = engine_for(config, tensors, dtype, kv_tokens=320, page_size=16)
    compare(replay(engine, tail_steps(requests, tail=45)), want, TOL[name, dtype], f"{name} {dtype} tail")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_down_to_two_tokens(models, name, dtype):
    config, tensors, requests, want = models[name, dtype]
    engine = engine_for(config, tensors, dtype, kv_tokens=320, page_size=8)
    compare(replay(engine, portion_steps(requests)), want, TOL[name, dtype], f"{name} {dtype} portions")
    compare(replay(engine, portion_steps(requests, sizes=(2, 2, 5, 24, 1, 3))), want, TOL[name, dtype], f"{name} {dtype} portions'")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_mixed_batches_with_pages_and_slots_used_again(models, name, dtype):
    """Four live requests at most in a pool that holds far fewer tokens than all requests together: every page and
    slot is given back and taken again (a slot's states start from zero again), portions run beside single tokens, and
    each row equals the request alone."""
    config, tensors, requests, want = models[name, dtype]
    builder, peak = mixed_steps(requests, seed=3, max_live=4)
    engine = engine_for(config, tensors, dtype, kv_tokens=peak, page_size=16, max_requests=4)
    compare(replay(engine, builder), want, TOL[name, dtype], f"{name} {dtype} mixed")
    assert engine.cache.used_tokens == 0
    assert engine.cache.high_water_tokens <= peak
    if dtype == "float32":
        # what else is in the batch and how a prompt was cut changes a row in 32-bit by rounding only (a split of the keys, and
        # a single token's read-out, add a row's terms in another order)
        alone = replay(engine_for(config, tensors, dtype, kv_tokens=320), whole_steps(requests))
        again = replay(engine, builder)
        for r in requests:
            for p in again[r]:
                assert (again[r][p] - alone[r][p]).abs().max().item() < TOL[name, dtype] / 2, (r, p)


def test_a_windowed_layer_gives_its_pages_back(models):
    """A request of 300 tokens in a model whose paged layer sees 100 keys and 33 first ones: the pool holds far fewer tokens than
    the request, the pages between the first keys and the window come back."""
    config, tensors, requests, want = models["C", "float32"]
    long = {"r6": requests["r6"]}
    engine = engine_for(config, tensors, "float32", kv_tokens=208, page_size=8, max_context=512)
    got = replay(engine, portion_steps(long, sizes=(16, 3, 9, 2, 40)))
    compare(got, {"r6": want["r6"]}, FLOAT32_TOL, "C in a small pool")
    assert engine.cache.high_water_tokens <= 208


def test_slots_of_finished_requests_start_again(models):
    """Ten requests through two slots: a slot's memory and its maximum start from zero for each."""
    config, tensors, _, _ = models["A", "float32"]
    requests = random_requests(config, [9, 30, 4, 17, 22, 3, 12, 40, 2, 25], 21)
    reference = plain_tensors(tensors)
    want = {r: plain.forward(config, reference, t).float() for r, t in requests.items()}
    builder, peak = mixed_steps(requests, seed=5, max_live=2)
    engine = engine_for(config, tensors, "float32", kv_tokens=peak, max_requests=2)
    compare(replay(engine, builder), want, FLOAT32_TOL, "A through two slots")


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_greedy_generation_through_the_scheduler(models, name):
    from damendaemon_b200.runtime import Runtime
    config, tensors, requests, _ = models[name, "float32"]
    reference = plain_tensors(tensors)
    prompts = [requests[r] for r in ("r1", "r2", "r5")]

    def greedy(prompt, n):
        ids = list(prompt)
        for _ in range(n):
            ids.append(int(plain.forward(config, reference, ids)[-1].argmax()))
        return ids[len(prompt):]
    want = [greedy(p, 12) for p in prompts]
    for graph in (False, True):
        runtime = Runtime(None, 512, config=config, tensors=tensors, dtype="float32", max_batch=4, page_size=16, use_graph=graph)
        assert runtime.generate_batch(prompts, 12, ignore_eos=True) == want
        assert runtime.engine.cache.used_tokens == 0
    reference = plain_tensors(models[name, "bfloat16"][1])
    want = [greedy(p, 12) for p in prompts]
    runtime = Runtime(None, 512, config=config, tensors=models[name, "bfloat16"][1], dtype="bfloat16", max_batch=4)
    got = runtime.generate_batch(prompts, 12, ignore_eos=True)
    for p, g, w in zip(prompts, got, want):
        if g != w:   # rounding may flip a near-tie; then the plain logits at the flip must be a near-tie
            i = next(i for i in range(12) if g[i] != w[i])
            row = plain.forward(config, reference, p + w[:i])[-1]
            assert abs(float(row[g[i]] - row[w[i]])) < max(0.15, 4.0 * abs(TOL[name, "bfloat16"]))


def test_long_decoding_in_a_graph(models):
    """Two hundred single-token steps of two requests, replayed from a CUDA graph after the first ones: the window
    passes many times over, the memories and their maxima are carried two hundred times."""
    from damendaemon_b200.engine import StepEntry
    config, tensors, _, _ = models["A", "float32"]
    requests = random_requests(config, [210, 190], 5)
    reference = plain_tensors(tensors)
    want = {r: plain.forward(config, reference, t).float() for r, t in requests.items()}
    engine = engine_for(config, tensors, "float32", kv_tokens=512, use_graph=True)
    assert engine.use_graph
    engine.step([StepEntry(r, t[:8], []) for r, t in requests.items()])
    for i in range(8, 190):
        logits = engine.step([StepEntry(r, t[i:i + 1], [0]) for r, t in requests.items()]).cpu()
        for row, r in zip(logits, requests):
            assert (row - want[r][i]).abs().max().item() < FLOAT32_TOL, (r, i)
    assert engine.graph_replays > 150


def test_the_replay_program_reads_this_architecture(models, tmp_path):
    import json
    import subprocess
    import sys

    import numpy as np

    from damendaemon_b200.weights import write_safetensors
    from trace_tools import ROOT
    config, tensors, requests, want = models["B", "float32"]
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(config))
    write_safetensors(folder / "model.safetensors", tensors)
    builder = portion_steps({"r6": requests["r6"]}, sizes=(9, 2, 30))
    text = "".join(json.dumps(s) + "\n" for s in builder.steps)
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32",
                           "--out", str(out), "--max-tokens", "128"], input=text, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-3000:]
    for s in builder.steps:
        rows = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, config["vocab"])
        for (r, p), row in zip(builder.where[s["step"]], rows):
            assert np.abs(row - want[r][p].numpy()).max() < FLOAT32_TOL


def test_the_command_line_makes_and_runs_a_model_of_this_architecture(tmp_path):
    """init-random writes a folder from the architecture's own config.json; run generates from it, greedy tokens equal
    to the plain implementation reading the same folder."""
    import json
    import subprocess
    import sys

    from trace_tools import ROOT
    cfg = tmp_path / "c.json"
    cfg.write_text(json.dumps(CONFIGS["D"]))
    made = subprocess.run([sys.executable, "-m", "damendaemon_b200", "init-random", str(cfg), str(tmp_path / "m"), "--seed", "4",
                           "--dtype", "float32"], capture_output=True, text=True, cwd=ROOT, timeout=600)
    assert made.returncode == 0 and (tmp_path / "m" / "model.safetensors").is_file(), made.stderr[-2000:]
    out = subprocess.run([sys.executable, "-m", "damendaemon_b200", "run", str(tmp_path / "m"), "--prompt-ids", "3,1,4,1,5,9,2,6",
                          "--max-tokens", "6", "--dtype", "float32", "--ignore-eos", "--context", "64"],
                         capture_output=True, text=True, cwd=ROOT, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    config, tensors = plain.read_folder(tmp_path / "m")
    ids = [3, 1, 4, 1, 5, 9, 2, 6]
    for _ in range(6):
        ids.append(int(plain.forward(config, tensors, ids)[-1].argmax()))
    assert [int(t) for t in out.stdout.split()] == ids[8:]
