"""Whole Sidalorn models (small random ones) through the framework's loader, step function, sequence slots and scheduler,
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
from oracle.stack_oracle import SidalornOracle  # noqa: E402

pytestmark = pytest.mark.gpu

# of the largest logit; a lost key, state, sink or filter tap moves logits by several per cent
TOL = {"float32": 1e-4, "bfloat16": 1e-2}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            cfg = SC.SIDALORN[name]
            w = SC.sidalorn_weights(cfg, seed=sum(map(ord, name)))
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
@pytest.mark.parametrize("name", sorted(SC.SIDALORN))
def test_prompt_portions_and_tokens(nat, folder, name, dtype):
    path, cfg, w = folder(name)
    rng = np.random.default_rng(1)
    oracle, layers = SidalornOracle(cfg, w), []
    tokens = SC.clear_tokens(oracle, 300, rng)
    want = oracle.step(tokens, layers)
    m = models.load(nat, path, dtype=dtype, sequences=2, max_len=310, max_rows=256)   # 300 rows: two passes
    s = m.acquire()
    o = m.step([(s, tokens[:200])], range(200), trace_layers=True)
    for i, x in enumerate(layers):
        check(o["layers"][i], x[:200], dtype, f"residual after layer {i}")
    check(o["logits"], want[:200], dtype, "prompt")
    check(m.step([(s, tokens[200:])], range(100))["logits"], want[200:], dtype, "rest in one step")
    m.release(s)
    for portions in ([300], [1], [2], [2, 97, 16, 3, 128, 1], [63, 2, 1, 1]):
        s = m.acquire()
        check(run_portions(m, s, tokens, portions), want, dtype, f"portions {portions}")
        assert m.length(s) == 300
        m.release(s)
    s = m.acquire()
    some = [0, 1, 63, 64, 127, 128, 255, 256, 299]
    check(m.step([(s, tokens)], some)["logits"], want[some], dtype, "wanted rows across passes")
    m.close()
    nat.free_all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["tiles", "wide_heads", "unaligned"])
def test_batches_of_unequal_requests(nat, folder, name, dtype):
    """Prompts, portions and decode rows of different sequences share a step; slots are freed and used again."""
    path, cfg, w = folder(name)
    rng = np.random.default_rng(2)
    m = models.load(nat, path, dtype=dtype, sequences=3, max_len=200)
    toks = {k: SC.clear_tokens(SidalornOracle(cfg, w), n, rng) for k, n in {"a": 180, "b": 33, "c": 5, "d": 160}.items()}
    want = {k: SidalornOracle(cfg, w).step(t) for k, t in toks.items()}
    slot, at = {}, dict.fromkeys(toks, 0)
    for step in ([("a", 40)], [("a", 1), ("b", 30)], [("b", 1), ("a", 117), ("c", 4)], [("c", 1), ("b", 1), ("a", 1)],
                 [("a", 20), ("b", 1), ("d", 2)], [("a", 1), ("d", 156)], [("d", 2)]):
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
    o, out = SidalornOracle(cfg, w), []
    logits, gaps = o.step(prompt)[-1], []
    for _ in range(n):
        top = np.sort(logits)[::-1]
        gaps.append(top[0] - top[1])
        out.append(int(np.argmax(logits)))
        logits = o.step([out[-1]])[-1]
    return out, gaps


@pytest.mark.parametrize("name", ["tiles", "recurrent"])
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
    m.close()
    nat.free_all()


@pytest.mark.parametrize("name", sorted(SC.SIDALORN))
def test_long_decoding_matches_one_prompt(nat, folder, name):
    """Tokens generated by graph replay for two sequences, fed again as one prompt each: the last step's logits agree."""
    path, cfg, w = folder(name)
    for dtype in ("float32", "bfloat16"):
        m = models.load(nat, path, dtype=dtype, sequences=3, max_len=700)
        starts, slots = ([5, 9, 2], [7] * 40), [m.acquire(), m.acquire()]
        first = [int(m.step([(s, p)], [len(p) - 1], want_next=True)["next"][0]) for s, p in zip(slots, starts)]
        m.begin_sequences(slots, first)
        ids, logits = m.generate(600, want_logits=True)
        for j, (s, p) in enumerate(zip(slots, starts)):
            t = m.acquire()
            fed = [*p, first[j]] + ids[:-1, j].tolist()
            again = m.step([(t, fed)], [len(fed) - 1])["logits"]
            assert m.length(s) == m.length(t)
            check(logits[j:j + 1], again, dtype, f"{dtype} after {len(fed)} tokens")
            m.release(t)
        m.close()
        nat.free_all()


def test_a_far_token_shows(nat, folder):
    """Sharp scores: a single key takes most of an attention's weight, often a far one. In 32-bit, in prompts and in decoding."""
    _, cfg, w = folder("tiles")
    w = dict(w)
    for i in (0, 2):
        w[f"l{i}.mix.uk"] = w[f"l{i}.mix.uk"] * 8.0      # sharp scores: a single key takes most of the weight
    rng = np.random.default_rng(7)
    path = SC.write_model(os.path.join(str(folder("tiles")[0]), "sharp"), cfg, w)
    m = models.load(nat, path, dtype="float32", sequences=1, max_len=700)
    for _ in range(2):
        tokens = rng.integers(0, cfg["vocab"], 650)
        want = SidalornOracle(cfg, w).step(tokens)
        s = m.acquire()
        got = np.concatenate([m.step([(s, tokens[:640])], range(640))["logits"]] +
                             [m.step([(s, [t])], [0])["logits"] for t in tokens[640:]])
        check(got, want, "float32", "sharp scores")
        m.release(s)
    m.close()
    nat.free_all()


def test_command_lines(folder, tmp_path):
    path, cfg, w = folder("tiles")
    rng = np.random.default_rng(4)
    a, b = rng.integers(0, cfg["vocab"], 20).tolist(), rng.integers(0, cfg["vocab"], 7).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:12], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[12:], "want": [7, 0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": b, "want": [6]}], "end": ["b"]}]
    run = os.path.join(helpers.ROOT, "bin", "trace_run")
    p = subprocess.run([run, "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "40"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    got = np.fromfile(tmp_path / "1.f32", "<f4").reshape(2, cfg["vocab"])
    check(got, SidalornOracle(cfg, w).step(a)[[19, 12]], "float32", "traced request a")
    check(np.fromfile(tmp_path / "2.f32", "<f4")[None], SidalornOracle(cfg, w).step(b)[-1:], "float32", "traced request b")
    p = subprocess.run([sys.executable, os.path.join(helpers.ROOT, "bin", "generate"), "--model", path, "--dtype", "float32",
                        "--max-new", "4", ",".join(map(str, a)), ",".join(map(str, b))], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    lines = [json.loads(x) for x in p.stdout.splitlines() if x.startswith("[")]
    assert lines == [greedy(cfg, w, a, 4)[0], greedy(cfg, w, b, 4)[0]]
