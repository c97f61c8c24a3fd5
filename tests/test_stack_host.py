"""CPU side of the layer-stack models: registry and configuration, weight files, rotation tables, the scheduler on a fake
model, and the plain oracle's own consistency."""
import json
import math
import struct

import numpy as np
import pytest

import helpers
import stack_cases as SC

helpers.load_package()
from m40_llm_b200 import models, weights as wt  # noqa: E402
from m40_llm_b200.engine import Engine  # noqa: E402
from m40_llm_b200.models.stack import rotary_tables  # noqa: E402
from oracle import stack_oracle as S  # noqa: E402


def test_registry_and_order():
    assert "Lamutar" in models.architectures()
    spec = models.read_config(SC.CASES["loop_tiles"])
    assert spec.order() == [("layer", 0), ("join", 0), ("layer", 1), ("layer", 2), ("join", 1), ("layer", 1), ("layer", 2),
                            ("join", 2), ("layer", 1), ("layer", 2), ("layer", 3)]
    assert models.read_config(SC.CASES["odd_sizes"]).order() == [("layer", 0), ("layer", 1), ("layer", 2)]
    assert models.read_config(SC.CASES["odd_sizes"]).soft_cap == 0.0
    with pytest.raises(ValueError, match="architecture"):
        models.read_config({"architecture": "Nothing"})
    bad = json.loads(json.dumps(SC.CASES["odd_sizes"]))
    bad["layers"][0]["type"] = "convolution"
    with pytest.raises(ValueError, match="unknown type"):
        models.read_config(bad)
    bad = json.loads(json.dumps(SC.CASES["loop_tiles"]))
    bad["loop"]["stop"] = 9
    with pytest.raises(ValueError, match="loop"):
        models.read_config(bad)


def test_weight_file_round_trip(tmp_path):
    p = str(tmp_path / "w.safetensors")
    a = np.array([[1.0, -2.5, 3.0]], np.float32)
    wt.write(p, {"a": a, "alpha": np.float32(0.5), "ids": np.array([3, -1], np.int32)})
    f = wt.TensorFile(p)
    assert f.shape("a") == (1, 3) and f.shape("alpha") == () and "b" not in f
    assert np.array_equal(f.f32("a"), a) and f.f32("alpha").reshape(-1)[0] == 0.5
    assert f.raw("ids")[1] == "I32" and list(f.raw("ids")[0]) == [3, -1]
    with pytest.raises(KeyError):
        f.raw("b")
    with open(p, "r+b") as h:      # a header longer than the file
        h.write(struct.pack("<Q", 1 << 40))
    with pytest.raises(ValueError):
        wt.TensorFile(p)


def test_bf16_rounding():
    x = np.array([1.0, 1.00390625, 1.01171875, -3.0e-39, 65504.0], np.float32)
    assert list(wt.bf16_to_f32(wt.f32_to_bf16(x))[:3]) == [1.0, 1.0, 1.015625]   # ties to even
    y = wt.bf16_to_f32(wt.f32_to_bf16(np.random.default_rng(0).standard_normal(1000).astype(np.float32)))
    assert np.array_equal(wt.bf16_to_f32(wt.f32_to_bf16(y)), y)


@pytest.mark.parametrize("base,dims", [(10000.0, 64), (1e6, 32), (500.0, 10), (2.0, 4)])
@pytest.mark.parametrize("scaling", [None, SC.YARN, {"factor": 32.0, "original": 4096, "fast": 32.0, "slow": 1.0},
                                     {"factor": 2.0, "original": 8, "fast": 1.0, "slow": 1.0}])
def test_rotation_tables(base, dims, scaling):
    turns, amp = rotary_tables(base, dims, scaling)
    f, a = S.rope_freqs(base, dims, scaling)
    assert np.allclose(turns * 2 * math.pi, f, rtol=1e-12) and amp == pytest.approx(a)
    plain = base ** (-2.0 * np.arange(dims // 2) / dims)
    if scaling is None:
        assert np.allclose(f, plain) and a == 1.0
    else:   # every frequency lies between the slowed one and its own
        assert (f <= plain * (1 + 1e-12)).all() and (f >= plain / scaling["factor"] * (1 - 1e-12)).all()


def test_yarn_by_hand():
    # dims 8, base 16: pair i turns at 16^(-i/4) = 2^-i; pair_with(t) = 8 ln(o / 2 pi t) / (2 ln 16)
    o = 2 * math.pi * 16.0
    f, a = S.rope_freqs(16.0, 8, {"factor": 2.0, "original": o, "fast": 8.0, "slow": 2.0})   # lo = 1, hi = 3
    assert np.allclose(f, [1.0, 0.5, 0.25 * (0.5 * 0.5 + 0.5), 0.125 * 0.5])
    assert a == pytest.approx(0.1 * math.log(2.0) + 1.0)


def test_oracle_rotated_values_are_relative():
    """Turning a value at its own position and the output back leaves only the distance between the two."""
    f = S.rope_freqs(100.0, 6)[0]
    v = np.random.default_rng(0).standard_normal((1, 1, 6))
    for shift in (0, 7):
        back = S.rotate_half(S.rotate_half(v, [3 + shift], f), [5 + shift], f, sign=-1.0)
        assert np.allclose(back, S.rotate_half(v, [2], f, sign=-1.0))


@pytest.mark.parametrize("name", sorted(SC.CASES))
def test_oracle_portions_agree(name):
    cfg = SC.CASES[name]
    w = SC.random_weights(cfg, 1)
    t = np.random.default_rng(1).integers(0, cfg["vocab"], 20)
    m = S.StackOracle(cfg, w)
    whole = m.step(t)
    m.reset()
    assert np.allclose(np.concatenate([m.step(t[:7]), m.step(t[7:9]), m.step(t[9:])]), whole, atol=1e-9)


def test_oracle_delta_rule_by_hand():
    """One head, one channel pair: the state after two tokens, written out."""
    eye = np.eye(2)
    h = np.array([[1.0, 2.0], [0.5, -1.0]])
    w = {n: eye for n in "rkvga"} | {"w1": np.zeros((1, 2)), "w2": np.zeros((2, 1)), "w0": np.array([0.0, 1.0]),
                                    "a.b": np.array([0.3, -0.2]), "norm": np.ones(2), "o": eye}
    _, st = S.general_delta(h, np.zeros((1, 2, 2)), w, {"heads": 1, "dim": 2}, 1e-5)
    decay = [math.exp(-math.exp(-0.5) / (1 + math.exp(-x))) for x in (0.0, 1.0)]
    a = [1 / (1 + math.exp(-(0.5 + 0.3))), 1 / (1 + math.exp(-(-1.0 - 0.2)))]
    u = [x / math.sqrt(1.25 + 1e-6) for x in (0.5, -1.0)]
    first = [[1.0, 2.0], [2.0, 4.0]]
    for i in range(2):
        for j in range(2):
            read = u[0] * first[0][j] + u[1] * first[1][j]
            assert st[0, i, j] == pytest.approx(decay[i] * first[i][j] - a[i] * u[i] * read + h[1][i] * h[1][j])


class FakeModel:
    """Next token = (sum of the sequence so far) % 97; checks what the scheduler hands over."""
    sequences = 2

    def __init__(self):
        self.seq, self.steps = {}, []
        self.free = [0, 1]

    def acquire(self):
        s = self.free.pop(0)
        self.seq[s] = []
        return s

    def release(self, s):
        del self.seq[s]
        self.free.append(s)

    def length(self, s):
        return len(self.seq[s])

    def step(self, entries, want=(), want_logits=True, want_next=False):
        nxt, rows = [], []
        for s, toks in entries:
            for t in toks:
                self.seq[s].append(int(t))
                rows.append(sum(self.seq[s]) % 97)
        self.steps.append([(s, len(t)) for s, t in entries])
        return {"next": np.array([rows[i] for i in want], np.uint32)}

    def begin_sequences(self, seqs, tokens):
        self.cur = list(zip(seqs, tokens))

    def generate(self, n):
        out = np.zeros((n, len(self.cur)), np.uint32)
        for i in range(n):
            for j, (s, t) in enumerate(self.cur):
                self.seq[s].append(int(t))
                out[i, j] = sum(self.seq[s]) % 97
                self.cur[j] = (s, out[i, j])
        return out, None


def test_scheduler_on_a_fake_model():
    def want(prompt, n, stop=None):
        seq, out = list(prompt), []
        while len(out) < n and not (out and out[-1] == stop):
            out.append(sum(seq) % 97)
            seq.append(out[-1])
        return out
    m = FakeModel()
    e = Engine(m, portion=8, burst=4)
    jobs = {e.submit(p, n, stop): (p, n, stop) for p, n, stop in
            (([1, 2, 3], 9, None), (list(range(30)), 5, None), ([4], 1, None), ([7] * 9, 30, 42), ([5, 6], 12, None))}
    out = e.run()
    assert {i: len(o) > 0 for i, o in out.items()} == dict.fromkeys(jobs, True)
    for i, (p, n, stop) in jobs.items():
        assert out[i] == want(p, n, stop), i
    assert not m.seq and sorted(m.free) == [0, 1]
    assert max(sum(n for _, n in s) for s in m.steps) <= 8 + 2        # a portion plus the decode rows
    with pytest.raises(ValueError):
        e.submit([], 3)


# ------------------------------------------------------------------------------------------------------- Sidalorn
def test_sidalorn_registry():
    assert "Sidalorn" in models.architectures()
    spec = models.read_config(SC.SIDALORN["tiles"])
    assert (spec.width, spec.vocab, spec.taps, spec.groups) == (192, 210, 4, 3)
    for at, key, bad, msg in ((("layers", 0), "type", "convolution", "unknown type"),
                              (("layers", 0, "mlp"), "kind", "sparse", "unknown feed-forward"), (("norm",), "groups", 7, "do not divide")):
        cfg = json.loads(json.dumps(SC.SIDALORN["tiles"]))
        d = cfg
        for k in at:
            d = d[k]
        d[key] = bad
        with pytest.raises(ValueError, match=msg):
            models.read_config(cfg)


@pytest.mark.parametrize("name", sorted(SC.SIDALORN))
def test_sidalorn_oracle_portions_agree(name):
    cfg = SC.SIDALORN[name]
    w = SC.sidalorn_weights(cfg, 1)
    t = np.random.default_rng(1).integers(0, cfg["vocab"], 20)
    m = S.SidalornOracle(cfg, w)
    whole = m.step(t)
    m.reset()
    assert np.allclose(np.concatenate([m.step(t[:7]), m.step(t[7:9]), m.step(t[9:10]), m.step(t[10:])]), whole, atol=1e-9)


def test_oracle_grouped_and_polynomial_norms_by_hand():
    x = np.array([[3.0, 4.0, 0.0, 2.0]])
    got = S.group_rms_norm(x, np.array([1.0, 2.0, 1.0, 1.0]), 0.5, 2)
    a, b = math.sqrt(12.5 + 0.5), math.sqrt(2.0 + 0.5)
    assert np.allclose(got, [[3 / a, 8 / a, 0.0, 2 / b]])
    z = np.array([[1.0, -2.0]])
    n = [math.sqrt(5 / 2 + 0.1), math.sqrt(17 / 2 + 0.1), math.sqrt(65 / 2 + 0.1)]
    assert np.allclose(S.poly_norm(z, (2.0, 3.0, 5.0, 7.0), 0.1),
                       [[2 / n[0] + 3 / n[1] + 5 / n[2] + 7, -4 / n[0] + 12 / n[1] - 40 / n[2] + 7]])


def test_oracle_convolution_by_hand():
    w = np.array([[2.0, 3.0, 5.0]])
    out, past = S.causal_conv(np.array([[1.0], [10.0], [100.0]]), np.zeros((2, 1)), w)
    assert out.ravel().tolist() == [5.0, 53.0, 532.0] and past.ravel().tolist() == [10.0, 100.0]
    out, past = S.causal_conv(np.array([[7.0]]), past, w, np.array([1.0]))
    assert out.ravel().tolist() == [20.0 + 300.0 + 35.0 + 1.0] and past.ravel().tolist() == [100.0, 7.0]


def test_oracle_recurrence_by_hand():
    one = lambda v: np.array([v])
    w = {"y": np.array([[1.0]]), "y.b": one(0.5), "x": np.array([[2.0]]), "x.b": one(0.0), "conv": np.array([[1.0]]), "conv.b": one(0.0),
         "ra": np.array([[[0.3]]]), "ra.b": np.array([[0.1]]), "ri": np.array([[[-0.2]]]), "ri.b": np.array([[0.4]]), "lam": one(-1.0),
         "o": np.array([[1.0]])}
    s = 0.0
    for h in (0.7, -1.1):
        u = 2 * h
        r, i = 1 / (1 + math.exp(-(0.3 * u + 0.1))), 1 / (1 + math.exp(-(-0.2 * u + 0.4)))
        a = math.exp(-8 * r * math.log(1 + math.exp(-1.0)))
        s = a * s + math.sqrt(1 - a * a) * i * u
    out, S2, _ = S.rglru(np.array([[0.7], [-1.1]]), np.zeros(1), np.zeros((0, 1)), w, {"blocks": 1})
    assert S2[0] == pytest.approx(s) and out[1, 0] == pytest.approx(s * S.gelu_tanh(-0.6))


def test_oracle_sink_takes_weight_once():
    """Two equal keys and a sink with the same score: each gets a third, and the sink brings no value."""
    eye = np.eye(2)
    w = {"q": np.zeros((2, 2)), "dkv": eye, "dkv.norm": np.ones(2), "uk": eye, "uv": eye, "sink": np.zeros(1), "o": eye}
    out, C = S.latent_attention(np.array([[1.0, 1.0], [1.0, -1.0]]), np.zeros((0, 2)), w, {"heads": 1, "dim": 2, "vdim": 2, "scale": 5.0}, 0.0)
    assert np.allclose(out, [[0.5, 0.5], [2 / 3, 0.0]]) and C.shape == (2, 2)


def test_oracle_route_groups_and_weights():
    s = np.array([[0.1, 0.2, 0.3, 0.4]])
    ids, w = S.route(np.log(s), np.array([0.0, 0.0, -1.0, -1.0]), {"top": 1, "scale": 2.0})
    assert ids.tolist() == [[1]] and np.allclose(w, 2.0)
    r = {"top": 2, "scale": 1.0, "groups": {"count": 2, "keep": 1}}
    ids, w = S.route(np.log(s), np.array([0.31, 0.0, 0.0, 0.0]), r)      # the group of 0.41 wins over that of 0.4
    assert ids.tolist() == [[0, 1]] and np.allclose(w, [[1 / 3, 2 / 3]])
    assert S.choice_margin(np.log(s), np.array([0.31, 0.0, 0.0, 0.0]), r) == pytest.approx(0.01)
