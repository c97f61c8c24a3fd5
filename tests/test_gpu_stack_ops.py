"""The layer-stack mechanisms one by one through the C ABI, against the plain float64 statements of
oracle/stack_oracle.py: projections with norms and tails, rotary attention, the generalised delta rule."""
import ctypes as C

import numpy as np
import pytest

from helpers import load_package

load_package()
from m40_llm_b200 import native as N  # noqa: E402
from m40_llm_b200.models.stack import rotary_tables  # noqa: E402
from m40_llm_b200.weights import bf16_to_f32, f32_to_bf16  # noqa: E402
from oracle import stack_oracle as S  # noqa: E402

pytestmark = pytest.mark.gpu


def close(got, want, tol, what=""):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert np.isfinite(got).all(), what
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-6)
    assert err <= tol, f"{what}: {err:.3g} of the largest value (limit {tol:g})"


def no_status(nat):
    st = np.zeros(1, np.uint32)
    assert nat.lib.m40llm_context_take_device_status(nat.ctx, st.ctypes.data) == 0
    assert st[0] == 0, f"device status {st[0]}"


# --------------------------------------------------------------------------------------------------- projections
def run_linear(nat, x, w, wdt, rows, w2=None, bias=None, residual=None, pre=None, post=None, act=0, exact=0, cap=0.0, ldx=0):
    up = lambda a: None if a is None else nat.buf(np.ascontiguousarray(a, np.float32)).ptr
    conv = {N.DT_BF16: f32_to_bf16, N.DT_F16: lambda a: a.astype(np.float16), N.DT_F32: lambda a: a.astype(np.float32)}[wdt]
    n, k = w.shape
    out = nat.buf(np.asarray(residual, np.float32) if residual is not None else rows * n * 4)
    norm = lambda s: N.Norm() if s is None else N.Norm(s["kind"], s.get("eps", 0.0), s.get("alpha", 0.0), up(s.get("w")), up(s.get("b")))
    c = N.Linear(up(x), nat.buf(conv(w)).ptr, None if w2 is None else nat.buf(conv(w2)).ptr, out.ptr, up(bias),
                 out.ptr if residual is not None else None, norm(pre), norm(post), rows, k, n, ldx, wdt, act, exact, cap)
    rc = nat.lib.m40llm_linear_async(nat.ctx, C.byref(c), 1)
    assert rc == 0, rc
    nat.sync(1)
    got = out.download(np.float32, (rows, n))
    nat.free_all()
    no_status(nat)
    return got


def rounded(rng, wdt, *shape):
    a = (rng.standard_normal(shape) / np.sqrt(shape[-1])).astype(np.float32)
    if wdt == N.DT_BF16:
        return bf16_to_f32(f32_to_bf16(a))
    return a.astype(np.float16).astype(np.float32) if wdt == N.DT_F16 else a


@pytest.mark.parametrize("rows", [1, 2, 9, 40, 129, 300])
@pytest.mark.parametrize("n,k", [(130, 192), (7, 1048), (520, 64), (40, 24), (33, 50)])
@pytest.mark.parametrize("wdt,exact", [(N.DT_BF16, 0), (N.DT_F16, 0), (N.DT_BF16, 1), (N.DT_F32, 0)])
def test_linear_pre_post_residual_cap(nat, rows, n, k, wdt, exact):
    rng = np.random.default_rng(rows * 1000 + n + k)
    x = rng.standard_normal((rows, k)).astype(np.float32)
    w = rounded(rng, wdt, n, k)
    pre = dict(kind=N.NORM_DYT, alpha=0.7, w=1 + 0.2 * rng.standard_normal(k), b=0.3 * rng.standard_normal(k))
    post = dict(kind=N.NORM_DYT, alpha=1.3, w=1 + 0.2 * rng.standard_normal(n), b=0.3 * rng.standard_normal(n))
    bias, res = rng.standard_normal(n), rng.standard_normal((rows, n))
    tol = 6e-6 if exact or wdt == N.DT_F32 else 4e-5
    got = run_linear(nat, x, w, wdt, rows, bias=bias, residual=res, pre=pre, post=post, exact=exact)
    y = S.dyt_norm(S.dyt_norm(x, 0.7, pre["w"], pre["b"]) @ w.T.astype(np.float64) + bias, 1.3, post["w"], post["b"]) + res
    close(got, y, tol, "dyt pre/post, residual in place")
    got = run_linear(nat, x, w, wdt, rows, pre=dict(kind=N.NORM_RMS, eps=1e-3, w=pre["w"]), exact=exact, cap=0.5)
    close(got, S.soft_cap(S.rms_norm(x, pre["w"], 1e-3) @ w.T.astype(np.float64), 0.5), tol, "rms pre, cap")


@pytest.mark.parametrize("rows", [1, 3, 70, 150, 400])
@pytest.mark.parametrize("n,k", [(200, 192), (72, 1024), (33, 50), (9570, 136)])
@pytest.mark.parametrize("act,fn", [(N.ACT_GELU_TANH, S.gelu_tanh), (N.ACT_SILU, lambda z: z * S.sigmoid(z))])
def test_linear_gated(nat, rows, n, k, act, fn):
    rng = np.random.default_rng(rows + n)
    x = 2 * rng.standard_normal((rows, k)).astype(np.float32)
    for exact in (0, 1):
        w, w2 = rounded(rng, N.DT_BF16, n, k), rounded(rng, N.DT_BF16, n, k)
        pre = dict(kind=N.NORM_DYT, alpha=0.5)      # no weight, no shift
        got = run_linear(nat, x, w, N.DT_BF16, rows, w2=w2, pre=pre, act=act, exact=exact)
        h = np.tanh(0.5 * x.astype(np.float64))
        close(got, fn(h @ w.T.astype(np.float64)) * (h @ w2.T.astype(np.float64)), 3e-6 if exact else 6e-5, f"exact={exact}")


@pytest.mark.parametrize("rows", [1, 5, 64, 300])
def test_linear_row_pitch(nat, rows):
    rng = np.random.default_rng(rows)
    ld, k, n = 212, 64, 96
    x = rng.standard_normal((rows, ld)).astype(np.float32)
    w = rounded(rng, N.DT_BF16, n, k)
    got = run_linear(nat, x, w, N.DT_BF16, rows, pre=dict(kind=N.NORM_DYT, alpha=1.0), ldx=ld)
    close(got, np.tanh(x[:, :k].astype(np.float64)) @ w.T.astype(np.float64), 3e-5)


def test_linear_rejects(nat):
    b = nat.buf(64 * 64 * 4)
    mk = lambda **kw: N.Linear(x=b.ptr, w=b.ptr, out=b.ptr, rows=2, K=64, N=8, w_dtype=N.DT_BF16, **kw)
    call = lambda c: nat.lib.m40llm_linear_async(nat.ctx, C.byref(c), 1)
    assert call(mk(ldx=63)) == -2
    assert call(mk(act=9)) == -3
    assert call(mk(pre=N.Norm(N.NORM_RMS, 1e-5, 0.0, None, None))) == -4
    assert call(mk(post=N.Norm(N.NORM_RMS, 1e-5, 0.0, None, None))) == -4
    assert call(mk(post=N.Norm(N.NORM_POLY, 1e-5, 0.0, b.ptr, None))) == -4
    assert nat.lib.m40llm_linear_async(nat.ctx, C.byref(N.Linear()), 1) == -1
    nat.free_all()


# --------------------------------------------------------------------------------------------------- rows of a step
class Rows:
    """Segments [(sequence, first position, tokens)] as M40llmStepRows."""

    def __init__(self, nat, segments, mul=1, add=0, max_len=0):
        seq, pos, seg = [], [], []
        for s, p0, n in segments:
            seg += [len(seq), n, s, p0]
            seq += [s] * n
            pos += list(range(p0, p0 + n))
        u = lambda a: nat.buf(np.array(a, np.uint32)).ptr
        self.n, self.pos = len(seq), np.array(pos)
        self.c = N.StepRows(len(seq), len(segments), max(s[2] for s in segments), max_len, mul, add, u(seq), u(pos),
                            u(np.array(pos) + 1), u(seg))


# --------------------------------------------------------------------------------------------------- rotary attention
class Attn:
    """Rotary attention on packed projections, on the device and in the oracle's terms."""

    def __init__(self, nat, H, G, D, V, dims, f32, slots=3, max_len=400, base=1e4, scaling=None, scale=None, seed=0, norms=True,
                 turn_values=True, gate=True, mul=2, add=1):
        self.nat, self.H, self.G, self.D, self.V, self.eps = nat, H, G, D, V, 1e-4
        self.mul, self.add, self.gate = mul, add, gate
        rng = np.random.default_rng(seed)
        self.scale = D ** -0.5 if scale is None else scale
        self.qn = (1 + 0.3 * rng.standard_normal(H * D)).astype(np.float32) if norms else None
        self.kn = (1 + 0.3 * rng.standard_normal(G * D)).astype(np.float32) if norms else None
        self.f, self.amp = S.rope_freqs(base, dims, scaling)
        self.fv = S.rope_freqs(base, V)[0] if turn_values else None
        kt, amp = rotary_tables(base, dims, scaling)
        assert abs(amp - self.amp) < 1e-12
        self.kv = nat.lib.m40llm_kvcache_create_typed(nat.ctx, max_len, slots * mul, G, D, V, N.DT_F32 if f32 else N.DT_F16)
        assert self.kv
        self.tabs = (kt, rotary_tables(base, V, None)[0] if turn_values else None)
        self.K = {s: np.zeros((0, G, D)) for s in range(slots)}
        self.Vv = {s: np.zeros((0, G, V)) for s in range(slots)}

    def width(self):
        return self.H * self.D + self.G * (self.D + self.V) + (self.H if self.gate else 0)

    def device(self, packed, segments, max_len=0):
        nat = self.nat
        up = lambda a, t: None if a is None else nat.buf(np.ascontiguousarray(a, t)).ptr
        rows = Rows(nat, segments, self.mul, self.add, max_len)
        out = nat.buf(rows.n * self.H * self.V * 4)
        c = N.RotaryAttention(up(packed, np.float32), up(self.qn, np.float32), up(self.kn, np.float32), up(self.tabs[0], np.float64),
                              up(self.tabs[1], np.float64), out.ptr, packed.shape[1], self.H, len(self.tabs[0]), 1 if self.gate else 0,
                              self.eps, self.amp, self.scale)
        rc = nat.lib.m40llm_attention_rotary_async(nat.ctx, self.kv, C.byref(c), C.byref(rows.c))
        assert rc == 0, rc
        nat.sync(1)
        got = out.download(np.float32, (rows.n, self.H, self.V))
        nat.free_all()
        no_status(nat)
        return got

    def oracle(self, packed, segments):
        H, G, D, V = self.H, self.G, self.D, self.V
        at, outs = 0, []
        for s, p0, n in segments:
            x = packed[at:at + n].astype(np.float64)
            at += n
            pos = np.arange(p0, p0 + n)
            q, k, v, g = np.split(x, [H * D, H * D + G * D, H * D + G * (D + V)], axis=1)
            if self.qn is not None:
                q, k = S.rms_norm(q, self.qn, self.eps), S.rms_norm(k, self.kn, self.eps)
            q = S.rotate_half(q.reshape(n, H, D), pos, self.f, self.amp)
            k = S.rotate_half(k.reshape(n, G, D), pos, self.f, self.amp)
            v = v.reshape(n, G, V)
            if self.fv is not None:
                v = S.rotate_half(v, pos, self.fv)
            K = self.K[s] = np.concatenate([self.K[s][:p0], k])
            Vv = self.Vv[s] = np.concatenate([self.Vv[s][:p0], v])
            o = np.zeros((n, H, V))
            for t in range(n):
                for h in range(H):
                    sc = K[:p0 + t + 1, h // (H // G)] @ q[t, h] * self.scale
                    p = np.exp(sc - sc.max())
                    o[t, h] = p / p.sum() @ Vv[:p0 + t + 1, h // (H // G)]
            if self.fv is not None:
                o = S.rotate_half(o, pos, self.fv, sign=-1.0)
            if self.gate:
                o = o * S.sigmoid(g)[:, :, None]
            outs.append(o)
        return np.concatenate(outs)

    def both(self, packed, segments, tol, what, max_len=0):
        close(self.device(packed, segments, max_len), self.oracle(packed, segments), tol, what)

    def close(self):
        self.nat.lib.m40llm_kvcache_destroy(self.kv)


ATTN = [  # H, G, D, V, rotated dims, f32 cache
    (4, 2, 64, 64, 32, 0), (2, 2, 128, 128, 128, 0), (16, 1, 64, 64, 16, 0), (3, 1, 48, 80, 48, 0), (6, 3, 32, 16, 8, 0),
    (2, 1, 128, 64, 32, 0), (4, 2, 64, 64, 32, 1), (3, 3, 20, 12, 4, 1), (2, 1, 256, 192, 256, 1),
]
YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}


@pytest.mark.parametrize("H,G,D,V,dims,f32", ATTN)
def test_attention_portions_and_decode(nat, H, G, D, V, dims, f32):
    """Portions that end at, just before and just after every tile border, then token by token, in two interleaved slots."""
    a = Attn(nat, H, G, D, V, dims, f32, scaling=YARN, seed=H + D)
    rng = np.random.default_rng(1)
    tol = 3e-6 if f32 else 3e-3
    p0 = {0: 0, 2: 0}
    plan = [[(0, 63)], [(0, 2)], [(2, 17), (0, 1)], [(0, 62)], [(0, 1), (2, 111)], [(2, 3)], [(0, 1), (2, 1)], [(2, 1)], [(0, 1)],
            [(0, 70)], [(0, 1), (2, 1)]]
    for n_step, step in enumerate(plan):
        segs = []
        for s, n in step:
            segs.append((s, p0[s], n))
            p0[s] += n
        packed = rng.standard_normal((sum(n for _, n in step), a.width())).astype(np.float32)
        a.both(packed, segs, tol, f"step {n_step} {segs}", max_len=max(p0.values()) if n_step % 2 else 0)
    a.close()


@pytest.mark.parametrize("H,G,D,V,dims,f32", ATTN)
@pytest.mark.parametrize("portion", [1, 2, 40])
def test_attention_far_key_stands_out(nat, H, G, D, V, dims, f32, portion):
    """One key, anywhere in the cache, carries nearly all the weight: a lost, shifted or masked key shows at once."""
    a = Attn(nat, H, G, D, V, dims, f32, max_len=800, scale=3.0 / D ** 0.5 * 4.0, base=1e7, seed=3, norms=True)
    if a.qn is not None:
        a.qn[:] = np.tile(a.qn[:D], H)
        a.kn[:] = 1.0
    rng = np.random.default_rng(7)
    n = 200
    packed = rng.standard_normal((n, a.width())).astype(np.float32)
    a.both(packed, [(1, 0, n)], 1e-5 if f32 else 8e-3, "prompt")
    key = a.K[1].copy()
    pos = n
    for target in (0, 1, 62, 63, 64, 65, 126, 127, 128, 129, 191, 192, 199):
        row = rng.standard_normal((portion, a.width())).astype(np.float32)
        for h in range(H):   # the query of head h points at its stored key
            want = S.rotate_half(key[target:target + 1, h // (H // G)][:, None], [pos + portion - 1], a.f, 1.0, sign=-1.0)[0, 0]
            row[-1, h * D:(h + 1) * D] = 4.0 * want / a.qn[:D]
        got, exp = a.device(row, [(1, pos, portion)]), a.oracle(row, [(1, pos, portion)])
        close(got, exp, 1e-5 if f32 else 8e-3, f"target {target}")
        pos += portion
    a.close()


@pytest.mark.parametrize("norms,turn,gate", [(False, True, True), (True, False, True), (True, True, False), (False, False, False)])
@pytest.mark.parametrize("D,V,f32", [(64, 64, 0), (40, 24, 0), (64, 64, 1)])
def test_attention_optional_parts(nat, norms, turn, gate, D, V, f32):
    a = Attn(nat, 4, 2, D, V, 16, f32, norms=norms, turn_values=turn, gate=gate, seed=9, scaling=YARN)
    rng = np.random.default_rng(2)
    for segs in ([(0, 0, 33)], [(0, 33, 1)], [(1, 0, 5), (0, 34, 90)]):
        a.both(rng.standard_normal((sum(s[2] for s in segs), a.width())).astype(np.float32), segs, 3e-6 if f32 else 3e-3, str(segs))
    a.close()


def test_attention_slot_used_again(nat):
    a = Attn(nat, 4, 2, 64, 64, 32, 0, seed=4)
    rng = np.random.default_rng(5)
    a.both(10 * rng.standard_normal((150, a.width())).astype(np.float32), [(1, 0, 150)], 3e-3, "first owner")
    a.K[1], a.Vv[1] = a.K[1][:0], a.Vv[1][:0]
    a.both(rng.standard_normal((70, a.width())).astype(np.float32), [(1, 0, 70)], 3e-3, "next owner, prompt")
    a.both(rng.standard_normal((1, a.width())).astype(np.float32), [(1, 70, 1)], 3e-3, "next owner, decode")
    a.close()


def test_attention_rejects(nat):
    a = Attn(nat, 4, 2, 64, 64, 32, 0)
    b = nat.buf(1 << 16)
    rows = Rows(nat, [(0, 0, 1)])
    mk = lambda **kw: N.RotaryAttention(**{**dict(packed=b.ptr, k_turns=b.ptr, out=b.ptr, ld=1024, q_heads=4, k_pairs=16), **kw})
    call = lambda c: nat.lib.m40llm_attention_rotary_async(nat.ctx, a.kv, C.byref(c), C.byref(rows.c))
    assert call(mk(packed=None)) == -1
    assert call(mk(ld=511)) == -2
    assert call(mk(q_heads=3)) == -3
    assert call(mk(k_pairs=33)) == -3
    # a slot or position outside the cache: nothing is written, the status word says so
    bad = Rows(nat, [(99, 0, 1)], 2, 1)
    c = mk(ld=a.width())
    assert nat.lib.m40llm_attention_rotary_async(nat.ctx, a.kv, C.byref(c), C.byref(bad.c)) == 0
    nat.sync(1)
    st = np.zeros(1, np.uint32)
    assert nat.lib.m40llm_context_take_device_status(nat.ctx, st.ctypes.data) == 0 and st[0] & 2
    # the f16 entry points refuse a cache with other element or value sizes
    kv = nat.lib.m40llm_kvcache_create_typed(nat.ctx, 16, 1, 2, 64, 32, N.DT_F16)
    assert nat.lib.m40llm_attention_last_token_f32_gqa_async(nat.ctx, kv, 0, b.ptr, 4, 4, b.ptr) == -4
    nat.lib.m40llm_kvcache_destroy(kv)
    nat.free_all()
    a.close()


# --------------------------------------------------------------------------------------------------- delta rule
class Delta:
    def __init__(self, nat, H, D, R, slots=3, seed=0, mul=2, add=1, wdt=N.DT_BF16):
        self.nat, self.H, self.D, self.R, self.mul, self.add, self.wdt = nat, H, D, R, mul, add, wdt
        rng = np.random.default_rng(seed)
        HD = H * D
        self.w2 = rounded(rng, wdt, HD, R)
        self.w0 = rng.uniform(-6, 2, HD).astype(np.float32)
        self.ab = rng.standard_normal(HD).astype(np.float32)
        self.on = (1 + 0.3 * rng.standard_normal(HD)).astype(np.float32)
        self.st = nat.lib.m40llm_statecache_create(nat.ctx, slots * mul, H, D)
        assert self.st
        self.S = {s: np.zeros((H, D, D)) for s in range(slots)}

    def width(self):
        return 5 * self.H * self.D + self.R

    def device(self, packed, segments, split_low_rank=False):
        nat = self.nat
        up = lambda a: nat.buf(np.ascontiguousarray(a, np.float32)).ptr
        conv = f32_to_bf16 if self.wdt == N.DT_BF16 else (lambda a: a.astype(np.float16 if self.wdt == N.DT_F16 else np.float32))
        rows = Rows(nat, segments, self.mul, self.add)
        out = nat.buf(rows.n * self.H * self.D * 4)
        low = up(np.tanh(packed[:, 5 * self.H * self.D:].astype(np.float64)) @ self.w2.T) if split_low_rank else None
        c = N.DeltaRule(up(packed), nat.buf(conv(self.w2)).ptr, up(self.w0), up(self.ab), up(self.on), low, out.ptr, packed.shape[1],
                        self.R, self.wdt, -np.exp(-0.5), 1e-6, 1e-5)
        rc = nat.lib.m40llm_delta_rule_async(nat.ctx, self.st, C.byref(c), C.byref(rows.c))
        assert rc == 0, rc
        nat.sync(1)
        got = out.download(np.float32, (rows.n, self.H * self.D))
        nat.free_all()
        no_status(nat)
        return got

    def oracle(self, packed, segments):
        # the oracle takes projections of h: with h = the packed row, each projection is a selection matrix
        H, D, R = self.H, self.D, self.R
        HD, n = H * D, self.width()
        pick = lambda lo, hi: np.eye(n)[lo:hi]
        w = {x: pick(i * HD, (i + 1) * HD) for i, x in enumerate("rkvga")}
        w |= {"w1": pick(5 * HD, n), "w2": self.w2.astype(np.float64), "w0": self.w0, "a.b": self.ab, "norm": self.on, "o": np.eye(HD)}
        outs, at = [], 0
        for s, p0, t in segments:
            st = self.S[s] if p0 else np.zeros((H, D, D))
            y, self.S[s] = S.general_delta(packed[at:at + t], st, w, {"heads": H, "dim": D}, 1e-5)
            outs.append(y)
            at += t
        return np.concatenate(outs)

    def state(self, s):
        out = np.empty((self.H, self.D, self.D), np.float32)
        slot = s * self.mul + self.add
        assert self.nat.lib.m40llm_statecache_debug_read(self.nat.ctx, self.st, slot, out.ctypes.data) == 0
        return out

    def close(self):
        self.nat.lib.m40llm_statecache_destroy(self.st)


@pytest.mark.parametrize("H,D,R", [(2, 16, 8), (3, 20, 1), (1, 33, 40), (4, 64, 24), (2, 72, 5), (2, 96, 16), (1, 128, 64),
                                   (1, 150, 7), (1, 200, 300), (1, 256, 16)])
def test_delta_rule_portions_and_decode(nat, H, D, R):
    d = Delta(nat, H, D, R, seed=D)
    rng = np.random.default_rng(D + R)
    p0 = {0: 0, 2: 0}
    # portions around the 16- or 32-token staging, mixed segments, single tokens; the low-rank product inside or outside
    for i, step in enumerate([[(0, 15)], [(0, 2)], [(2, 16), (0, 1)], [(0, 1), (2, 1)], [(2, 17)], [(0, 33), (2, 2)], [(0, 1)], [(2, 1)],
                              [(0, 32)], [(2, 31), (0, 65)], [(2, 140)]]):
        segs = []
        for s, n in step:
            segs.append((s, p0[s], n))
            p0[s] += n
        packed = rng.standard_normal((sum(n for _, n in step), d.width())).astype(np.float32)
        close(d.device(packed, segs, split_low_rank=i % 2 == 1), d.oracle(packed, segs), 2e-5, f"step {i} {segs}")
    for s in (0, 2):
        close(d.state(s), d.S[s], 5e-6, f"state of slot {s}")
    d.close()


def test_delta_rule_prompt_equals_tokens_and_slot_reuse(nat):
    d = Delta(nat, 3, 40, 12, seed=5)
    rng = np.random.default_rng(6)
    packed = rng.standard_normal((90, d.width())).astype(np.float32)
    whole = d.device(packed, [(0, 0, 90)])
    whole_state = d.state(0)
    ones = np.concatenate([d.device(packed[t:t + 1], [(1, t, 1)]) for t in range(90)])
    close(ones, whole, 2e-6, "token by token")
    close(d.state(1), whole_state, 2e-6, "state")
    # the slot's next owner starts from zero, as a prompt and as a single token
    close(d.device(packed[:5], [(0, 0, 5)]), whole[:5], 2e-6, "slot used again, prompt")
    close(d.device(packed[:1], [(1, 0, 1)]), whole[:1], 2e-6, "slot used again, one token")
    d.close()


def test_delta_rule_long_memory(nat):
    """Slow decay and a removal rate near zero: what the first tokens wrote must still be read a thousand tokens later."""
    d = Delta(nat, 1, 48, 4, seed=8)
    d.w0[:], d.ab[:] = -12.0, -12.0
    d.w2[:] = 0.0
    rng = np.random.default_rng(9)
    n = 1000
    packed = 0.05 * rng.standard_normal((n, d.width())).astype(np.float32)
    HD = 48
    packed[:3, HD:2 * HD] *= 60.0          # three strong keys at the start ...
    packed[-1, :HD] = packed[1, HD:2 * HD]  # ... and a read-out that asks for the second
    close(d.device(packed, [(2, 0, n)]), d.oracle(packed, [(2, 0, n)]), 2e-5, "prompt")
    close(d.state(2), d.S[2], 1e-4, "state")      # a thousand equal f32 decays: their common rounding adds up
    d.close()


@pytest.mark.parametrize("wdt", [N.DT_F16, N.DT_F32])
def test_delta_rule_other_weight_types(nat, wdt):
    d = Delta(nat, 2, 32, 10, seed=2, wdt=wdt)
    packed = np.random.default_rng(3).standard_normal((20, d.width())).astype(np.float32)
    close(d.device(packed, [(0, 0, 20)]), d.oracle(packed, [(0, 0, 20)]), 2e-5)
    d.close()


def test_delta_rule_rejects(nat):
    d = Delta(nat, 2, 32, 10)
    b = nat.buf(1 << 14)
    rows = Rows(nat, [(0, 0, 1)])
    mk = lambda **kw: N.DeltaRule(**{**dict(packed=b.ptr, w2=b.ptr, w0=b.ptr, a_bias=b.ptr, norm=b.ptr, out=b.ptr, ld=330, rank=10,
                                            w_dtype=N.DT_BF16), **kw})
    call = lambda c: nat.lib.m40llm_delta_rule_async(nat.ctx, d.st, C.byref(c), C.byref(rows.c))
    assert call(mk(w0=None)) == -1 and call(mk(ld=329)) == -2 and call(mk(rank=0)) == -2 and call(mk(w_dtype=7)) == -3
    assert nat.lib.m40llm_statecache_create(nat.ctx, 1, 1, 257) is None
    nat.free_all()
    d.close()


def test_embed_concat_gather(nat):
    rng = np.random.default_rng(0)
    table = bf16_to_f32(f32_to_bf16(rng.standard_normal((9, 20))))
    ids = np.array([8, 0, 3], np.uint32)
    L = nat.lib
    out = nat.buf(3 * 40 * 4)
    for dt, raw in ((N.DT_BF16, f32_to_bf16(table)), (N.DT_F16, table.astype(np.float16)), (N.DT_F32, table)):
        assert L.m40llm_embed_tokens_async(nat.ctx, nat.buf(raw).ptr, dt, nat.buf(ids).ptr, out.ptr, 3, 20, 9) == 0
        nat.sync(1)
        want = table[ids] if dt != N.DT_F16 else table.astype(np.float16).astype(np.float32)[ids]
        assert np.array_equal(out.download(np.float32, (3, 20)), want)
    a, b = rng.standard_normal((2, 3, 20)).astype(np.float32)
    assert L.m40llm_concat_rows_async(nat.ctx, nat.buf(a).ptr, nat.buf(b).ptr, out.ptr, 3, 20) == 0
    nat.sync(1)
    assert np.array_equal(out.download(np.float32, (3, 40)), np.concatenate([a, b], 1))
    assert L.m40llm_gather_rows_async(nat.ctx, nat.buf(a).ptr, nat.buf(np.array([2, 0], np.uint32)).ptr, out.ptr, 2, 20, 3) == 0
    nat.sync(1)
    assert np.array_equal(out.download(np.float32, (2, 20)), a[[2, 0]])
    nat.free_all()
