"""Whole Lamutar models (small random ones) through the framework's loader, step function, sequence slots and scheduler,
against the plain float64 model of oracle/stack_oracle.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import helpers
import stack_cases as SC

helpers.load_package()
from m40_llm_b200 import models  # noqa: E402
from m40_llm_b200.engine import Engine  # noqa: E402
from oracle.stack_oracle import StackOracle  # noqa: E402

pytestmark = pytest.mark.gpu

# of the largest logit; a lost key, state or table entry moves logits by several per cent
TOL = {"float32": 1e-4, "bfloat16": 1e-2}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            cfg = SC.CASES[name]
            w = SC.random_weights(cfg, seed=sum(map(ord, name)))
            made[name] = (SC.write_model(tmp_path_factory.mktemp(name), cfg, w), cfg, w)
        return made[name]
    return get


def check(got, want, dtype, what):
    assert np.isfinite(got).all(), what
    err = np.abs(got - want).max() / np.abs(want).max()
    assert err <= TOL[dtype], f"{what}: {err:.3g}"


def run_portions(model, slot, tokens, portions):
    rows, at, i = [], 0, 0
    while at < len(tokens):
        n = min(portions[i % len(portions)], len(tokens) - at)
        rows.append(model.step([(slot, tokens[at:at + n])], range(n))["logits"])
        at += n
        i += 1
    return np.concatenate(rows)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SC.CASES))
def test_prompt_portions_and_tokens(nat, folder, name, dtype):
    path, cfg, w = folder(name)
    rng = np.random.default_rng(1)
    tokens = rng.integers(0, cfg["vocab"], 150)
    layers = []
    want = StackOracle(cfg, w).step(tokens, layers)
    m = models.load(nat, path, dtype=dtype, sequences=2, max_len=160, max_rows=128)   # 150 rows: two passes
    s = m.acquire()
    o = m.step([(s, tokens[:100])], range(100), trace_layers=True)
    check(o["logits"], want[:100], dtype, "prompt")
    for i, x in enumerate(layers):
        check(o["layers"][i], x[:100], dtype, f"residual after layer run {i}")
    check(m.step([(s, tokens[100:])], range(50))["logits"], want[100:], dtype, "rest in one step")
    m.release(s)
    for portions in ([150], [1], [2], [2, 37, 16, 3, 64, 1], [63, 2, 1]):
        s = m.acquire()
        check(run_portions(m, s, tokens, portions), want, dtype, f"portions {portions}")
        assert m.length(s) == 150
        m.release(s)
    # only the wanted rows, more than one logits pass
    s = m.acquire()
    some = [0, 1, 63, 64, 127, 128, 149]
    check(m.step([(s, tokens)], some)["logits"], want[some], dtype, "wanted rows across passes")
    m.close()
    nat.free_all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["loop_tiles", "odd_sizes"])
def test_batches_of_unequal_requests(nat, folder, name, dtype):
    """Prompts, portions and decode rows of different sequences share a step; slots are freed and used again."""
    path, cfg, w = folder(name)
    rng = np.random.default_rng(2)
    m = models.load(nat, path, dtype=dtype, sequences=3, max_len=100)
    toks = {k: rng.integers(0, cfg["vocab"], n) for k, n in {"a": 80, "b": 33, "c": 5, "d": 60}.items()}
    want = {k: StackOracle(cfg, w).step(t) for k, t in toks.items()}
    slot, at = {}, dict.fromkeys(toks, 0)
    for step in ([("a", 40)], [("a", 1), ("b", 30)], [("b", 1), ("a", 17), ("c", 4)], [("c", 1), ("b", 1), ("a", 1)],
                 [("a", 20), ("b", 1), ("d", 2)], [("d", 57), ("a", 1)], [("d", 1)]):
        entries, rows = [], []
        for k, n in step:
            if k not in slot:
                slot[k] = m.acquire()
            entries.append((slot[k], toks[k][at[k]:at[k] + n]))
            rows.append(want[k][at[k]:at[k] + n])
            at[k] += n
        total = sum(n for _, n in step)
        check(m.step(entries, range(total))["logits"], np.concatenate(rows), dtype, str(step))
        for k in list(slot):
            if at[k] == len(toks[k]):
                m.release(slot.pop(k))
    assert all(at[k] == len(t) for k, t in toks.items())
    m.close()
    nat.free_all()


def greedy(cfg, w, prompt, n):
    o, out = StackOracle(cfg, w), []
    logits, gaps = o.step(prompt)[-1], []
    for _ in range(n):
        top = np.sort(logits)[::-1]
        gaps.append(top[0] - top[1])
        out.append(int(np.argmax(logits)))
        logits = o.step([out[-1]])[-1]
    return out, gaps


@pytest.mark.parametrize("name", ["loop_tiles", "delta_only"])
def test_greedy_generation_through_the_scheduler(nat, folder, name):
    """More requests than slots, prompts cut into portions, graph-replayed bursts; 32-bit so that ids are comparable."""
    path, cfg, w = folder(name)
    rng = np.random.default_rng(3)
    m = models.load(nat, path, dtype="float32", sequences=2, max_len=140)
    engine = Engine(m, portion=24, burst=8)
    jobs = {}
    for n, new in ((30, 40), (3, 12), (50, 5), (1, 20)):
        prompt = rng.integers(0, cfg["vocab"], n).tolist()
        jobs[engine.submit(prompt, new)] = (prompt, new)
    out = engine.run()
    for i, (prompt, new) in jobs.items():
        want, gaps = greedy(cfg, w, prompt, new)
        first = next((t for t in range(new) if out[i][t] != want[t]), new)
        assert len(out[i]) == new
        assert first == new or gaps[first] < 1e-3, f"request {i}: token {first} of {new} differs, gap {gaps[first]}"
    assert m.graph_replays() > 0
    # all slots are free again, and a stop token ends a request
    engine = Engine(m, portion=16)
    prompt, new = jobs[min(jobs)]
    ids = out[min(jobs)]
    r = engine.submit(prompt, new, stop=ids[2])
    assert engine.run()[r] == ids[:ids.index(ids[2]) + 1]
    m.close()
    nat.free_all()


@pytest.mark.parametrize("name", ["loop_tiles", "unaligned"])
def test_long_decoding_matches_one_prompt(nat, folder, name):
    """Tokens generated by graph replay, fed again as one prompt: the last step's logits agree."""
    path, cfg, w = folder(name)
    for dtype in ("float32", "bfloat16"):
        m = models.load(nat, path, dtype=dtype, sequences=2, max_len=700)
        s = m.acquire()
        first = m.step([(s, [5, 9, 2])], [2], want_next=True)["next"]
        m.begin_sequences([s], first)
        ids, logits = m.generate(600, want_logits=True)
        t = m.acquire()
        fed = [5, 9, 2, int(first[0])] + ids[:-1, 0].tolist()
        again = m.step([(t, fed)], [len(fed) - 1])["logits"]
        assert m.length(s) == m.length(t)
        check(logits, again, dtype, f"{dtype} after {len(fed)} tokens")
        m.close()
        nat.free_all()


def test_step_errors(nat, folder):
    path, cfg, _ = folder("delta_only")
    m = models.load(nat, path, sequences=1, max_len=10)
    with pytest.raises(RuntimeError, match="step_entry"):
        m.step([(0, [1])])                     # not acquired
    s = m.acquire()
    with pytest.raises(RuntimeError, match="no free sequence slot"):
        m.acquire()
    with pytest.raises(RuntimeError, match="token_id"):
        m.step([(s, [cfg["vocab"]])])
    with pytest.raises(RuntimeError, match="too_long"):
        m.step([(s, [0] * 11)])
    with pytest.raises(RuntimeError, match="wanted_rows"):
        m.step([(s, [0, 1])], [2])
    with pytest.raises(RuntimeError, match="step_entry"):
        m.step([(s, [0]), (s, [1])])
    m.step([(s, [0] * 10)])
    m.release(s)
    with pytest.raises(RuntimeError):
        m.release(s)
    m.close()
    nat.free_all()


def test_command_lines(folder, tmp_path):
    path, cfg, w = folder("loop_tiles")
    rng = np.random.default_rng(4)
    a, b = rng.integers(0, cfg["vocab"], 20).tolist(), rng.integers(0, cfg["vocab"], 7).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:12], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[12:], "want": [7, 0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": b, "want": [6]}], "end": ["b"]}]
    run = os.path.join(helpers.ROOT, "bin", "trace_run")
    p = subprocess.run([run, "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "40"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (tmp_path / "0.f32").exists()
    got = np.fromfile(tmp_path / "1.f32", "<f4").reshape(2, cfg["vocab"])
    check(got, StackOracle(cfg, w).step(a)[[19, 12]], "float32", "traced request a")
    check(np.fromfile(tmp_path / "2.f32", "<f4")[None], StackOracle(cfg, w).step(b)[-1:], "float32", "traced request b")
    p = subprocess.run([sys.executable, os.path.join(helpers.ROOT, "bin", "generate"), "--model", path, "--dtype", "float32",
                        "--max-new", "4", ",".join(map(str, a)), ",".join(map(str, b))], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    lines = [json.loads(x) for x in p.stdout.splitlines() if x.startswith("[")]
    assert lines == [greedy(cfg, w, a, 4)[0], greedy(cfg, w, b, 4)[0]]
