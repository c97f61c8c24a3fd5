"""Sidalorn's mechanisms one by one through the C ABI, against the plain float64 statements of oracle/stack_oracle.py: grouped
and polynomial norms around projections, the short convolution, latent attention, the real-gated recurrence, the experts."""
import ctypes as C

import numpy as np
import pytest

from helpers import load_package

load_package()
from m40_llm_b200 import native as N  # noqa: E402
from m40_llm_b200.weights import bf16_to_f32, f32_to_bf16  # noqa: E402
from oracle import stack_oracle as S  # noqa: E402
from test_gpu_stack_ops import Rows, close, no_status, rounded, run_linear  # noqa: E402

pytestmark = pytest.mark.gpu


def b16(a):
    return bf16_to_f32(f32_to_bf16(np.asarray(a, np.float32)))


def f32(nat, a):
    return nat.buf(np.ascontiguousarray(a, np.float32)).ptr


def bits(nat, a):
    return nat.buf(f32_to_bf16(np.ascontiguousarray(a, np.float32))).ptr


# -------------------------------------------------------------------------------------------------- norms of projections
class Norms:
    """run_linear takes norms as dicts; this one carries groups and the activation too."""

    def __init__(self, nat):
        self.nat = nat

    def norm(self, kind, eps=0.0, w=None, groups=0, act=0):
        return N.Norm(kind, eps, 0.0, None if w is None else f32(self.nat, w), None, groups, act)

    def run(self, x, w, rows, pre=None, post=None, residual=None, exact=0, ldx=0, act=0):
        nat, (n, k) = self.nat, w.shape
        out = nat.buf(np.asarray(residual, np.float32) if residual is not None else rows * n * 4)
        c = N.Linear(f32(nat, x), bits(nat, w), None, out.ptr, None, out.ptr if residual is not None else None, pre or N.Norm(),
                     post or N.Norm(), rows, k, n, ldx, N.DT_BF16, act, exact, 0.0)
        assert nat.lib.m40llm_linear_async(nat.ctx, C.byref(c), 1) == 0
        nat.sync(1)
        got = out.download(np.float32, (rows, n))
        nat.free_all()
        no_status(nat)
        return got


@pytest.mark.parametrize("rows", [1, 2, 33, 300])
@pytest.mark.parametrize("n,k,groups", [(120, 192, 3), (96, 1000, 1), (520, 64, 40), (35, 50, 5), (64, 9000, 2)])
@pytest.mark.parametrize("exact", [0, 1])
def test_norms_around_a_projection(nat, rows, n, k, groups, exact):
    rng = np.random.default_rng(rows + n + k)
    t = Norms(nat)
    # parts of very different size: one root mean square for the whole row would be far off
    x = rng.standard_normal((rows, k)) * np.repeat(10.0 ** rng.uniform(-2, 2, n_parts(k, groups)), k // n_parts(k, groups))
    x = x.astype(np.float32)
    w = rounded(rng, N.DT_BF16, n, k)
    w64 = w.astype(np.float64)
    g_in, res = n_parts(k, groups), rng.standard_normal((rows, n))
    wk, wn = 1 + 0.3 * rng.standard_normal(k), 1 + 0.3 * rng.standard_normal(n)
    tol = 1e-5 if exact else 6e-5
    y = S.group_rms_norm(x, wk, 1e-4, g_in) @ w64.T
    close(t.run(x, w, rows, pre=t.norm(N.NORM_RMS, 1e-4, wk, g_in), exact=exact), y, tol, "grouped before")
    z = rng.standard_normal((rows, k)).astype(np.float32)
    y = S.group_rms_norm(z @ w64.T, wn, 1e-4, groups) + res
    close(t.run(z, w, rows, post=t.norm(N.NORM_RMS, 1e-4, wn, groups), residual=res, exact=exact), y, tol, "grouped after, residual")
    coef = np.array([0.7, -0.4, 0.3, -1.1], np.float32)
    y = S.poly_norm(z, coef, 1e-4) @ w64.T
    close(t.run(z, w, rows, pre=t.norm(N.NORM_POLY, 1e-4, coef), exact=exact), y, 3 * tol, "polynomial before")
    y = S.gelu_erf(z) @ w64.T
    close(t.run(z, w, rows, pre=t.norm(N.NORM_ACT, act=N.ACT_GELU_ERF), exact=exact), y, tol, "activation before")


def n_parts(k, groups):
    return groups if k % groups == 0 else 1


def test_polynomial_norm_of_a_padded_pitch(nat):
    rng = np.random.default_rng(5)
    t = Norms(nat)
    for rows in (1, 7):
        x, w = rng.standard_normal((rows, 104)).astype(np.float32), rounded(rng, N.DT_BF16, 40, 72)
        y = S.gelu_erf(x[:, :72]) @ w.astype(np.float64).T
        close(t.run(x, w, rows, pre=t.norm(N.NORM_ACT, act=N.ACT_GELU_ERF), ldx=104), y, 6e-5)


def test_exact_gelu_gate(nat):
    rng = np.random.default_rng(6)
    x, w, w2 = 2 * rng.standard_normal((5, 128)).astype(np.float32), rounded(rng, N.DT_BF16, 48, 128), rounded(rng, N.DT_BF16, 48, 128)
    got = run_linear(nat, x, w, N.DT_BF16, 5, w2=w2, act=N.ACT_GELU_ERF)
    close(got, S.gelu_erf(x @ w.T.astype(np.float64)) * (x @ w2.T.astype(np.float64)), 6e-5)


def test_norm_arguments(nat):
    b = nat.buf(64 * 64 * 4)
    call = lambda **kw: nat.lib.m40llm_linear_async(nat.ctx, C.byref(N.Linear(x=b.ptr, w=b.ptr, out=b.ptr, rows=2, K=64, N=8,
                                                                            w_dtype=N.DT_BF16, **kw)), 1)
    assert call(pre=N.Norm(N.NORM_RMS, 1e-5, 0.0, b.ptr, None, 7)) == -4      # 7 parts of 64
    assert call(pre=N.Norm(N.NORM_POLY, 1e-5, 0.0, None, None)) == -4
    assert call(pre=N.Norm(N.NORM_ACT, 0.0, 0.0, None, None, 0, 9)) == -4
    assert call(post=N.Norm(N.NORM_POLY, 1e-5, 0.0, b.ptr, None)) == -4
    nat.free_all()


# -------------------------------------------------------------------------------------------------- short convolution
@pytest.mark.parametrize("dim,taps,bias,add", [(200, 4, True, 0), (96, 3, False, 1), (130, 2, True, 1), (40, 1, False, 1),
                                               (33, 9, True, 0), (64, 32, False, 0)])
def test_short_convolution(nat, dim, taps, bias, add):
    rng = np.random.default_rng(dim + taps)
    w, b = rng.standard_normal((dim, taps)).astype(np.float32), rng.standard_normal(dim).astype(np.float32) if bias else None
    ring = nat.lib.m40llm_statecache_create_values(nat.ctx, 7, taps * dim)
    dw, db = f32(nat, w), f32(nat, b) if bias else None
    T = 150
    x = {s: rng.standard_normal((T, dim)).astype(np.float32) for s in range(3)}
    want = {s: S.causal_conv(v, np.zeros((taps - 1, dim)), w, b)[0] + add * v for s, v in x.items()}
    # sequences begin again in slots that hold old inputs; pieces of 1, 2 and more rows, several sequences together
    for plan in ([[(0, 150)]], [[(0, 1)]] * 40, [[(0, 2), (1, 33)], [(1, 1), (0, 1)], [(0, 70), (1, 3), (2, 1)], [(2, 2)], [(2, 100), (0, 5)]]):
        at = dict.fromkeys(x, 0)
        for step in plan:
            segs = [(s, at[s], n) for s, n in step]
            rows = Rows(nat, segs, mul=2, add=1)
            xin = np.concatenate([x[s][p:p + n] for s, p, n in segs])
            out = nat.buf(xin.size * 4)
            c = N.ShortConv(f32(nat, np.concatenate([xin, xin], axis=1)), dw, db, out.ptr, 2 * dim, dim, taps, add)
            assert nat.lib.m40llm_short_conv_async(nat.ctx, ring, C.byref(c), C.byref(rows.c)) == 0
            nat.sync(1)
            close(out.download(np.float32, xin.shape), np.concatenate([want[s][p:p + n] for s, p, n in segs]), 3e-6, str(step))
            for s, n in step:
                at[s] += n
    no_status(nat)
    bad = Rows(nat, [(3, 0, 1)], mul=2, add=1)      # slot 7 of 7
    if taps > 1:
        assert nat.lib.m40llm_short_conv_async(nat.ctx, ring, C.byref(c), C.byref(bad.c)) == 0
        st = np.zeros(1, np.uint32)
        nat.sync(1)
        nat.lib.m40llm_context_take_device_status(nat.ctx, st.ctypes.data)
        assert st[0] == 2
    nat.lib.m40llm_statecache_destroy(ring)
    nat.free_all()


# -------------------------------------------------------------------------------------------------- latent attention
class Latent:
    def __init__(self, nat, H, D, V, R, fp32, sink=True, scale=None, slots=5, max_len=1400, seed=0, sharp=1.0):
        self.nat, self.H, self.D, self.V, self.R, self.eps = nat, H, D, V, R, 1e-4
        rng = np.random.default_rng(seed)
        self.scale = D ** -0.5 if scale is None else scale
        self.cn = (1 + 0.3 * rng.standard_normal(R)).astype(np.float32)
        self.uk, self.uv = b16(sharp * rng.standard_normal((H * D, R)) / R ** 0.5), b16(rng.standard_normal((H * V, R)) / R ** 0.5)
        self.sink = rng.uniform(-1, 4, H).astype(np.float32) if sink else None
        self.kv = nat.lib.m40llm_kvcache_create_typed(nat.ctx, max_len, slots, 1, R, 0, N.DT_F32 if fp32 else N.DT_F16)
        self.ld = (H * D + R + 7) // 8 * 8
        ukt = self.uk.reshape(H, D, R).transpose(0, 2, 1).reshape(H * R, D)
        self.dev = [f32(nat, self.cn), bits(nat, self.uk), bits(nat, ukt), bits(nat, self.uv), f32(nat, self.sink) if sink else None]

    def oracle(self, q, c):
        """q [T, H * D], c [T, R] of one sequence from position 0 -> [T, H * V]."""
        eye = np.eye(self.H * self.D)
        w = {"q": np.concatenate([eye, np.zeros((self.H * self.D, self.R))], 1), "dkv.norm": self.cn, "uk": self.uk.astype(np.float64),
             "dkv": np.concatenate([np.zeros((self.R, self.H * self.D)), np.eye(self.R)], 1), "uv": self.uv.astype(np.float64),
             "sink": self.sink if self.sink is not None else np.full(self.H, -1e30), "o": np.eye(self.H * self.V)}
        m = {"heads": self.H, "dim": self.D, "vdim": self.V, "scale": self.scale}
        return S.latent_attention(np.concatenate([q, c], 1), np.zeros((0, self.R)), w, m, self.eps)[0]

    def run(self, segs, q, c, max_len=0, host=True):
        nat = self.nat
        rows = Rows(nat, segs, mul=2, add=1, max_len=max_len)
        if host:
            flat, at = [], 0
            for s, p0, n in segs:
                flat += [at, n, s, p0]
                at += n
            rows.host = np.array(flat, np.uint32)
            rows.c.seg_host = rows.host.ctypes.data
        packed = np.zeros((rows.n, self.ld), np.float32)
        packed[:, :self.H * self.D], packed[:, self.H * self.D:self.H * self.D + self.R] = q, c
        out = nat.buf(rows.n * self.H * self.V * 4)
        call = N.LatentAttention(f32(nat, packed), *self.dev, out.ptr, self.ld, self.H, self.D, self.V, N.DT_BF16, self.eps, self.scale)
        rc = nat.lib.m40llm_attention_latent_async(nat.ctx, self.kv, C.byref(call), C.byref(rows.c))
        assert rc == 0, rc
        nat.sync(1)
        return out.download(np.float32, (rows.n, self.H * self.V))

    def close(self):
        self.nat.lib.m40llm_kvcache_destroy(self.kv)
        self.nat.free_all()


LATENT = [(6, 64, 64, 128), (2, 128, 128, 512), (16, 64, 64, 64), (20, 32, 48, 80), (3, 96, 16, 256), (3, 10, 14, 21), (33, 16, 16, 48),
          (1, 128, 128, 1024), (5, 128, 64, 192), (40, 64, 64, 384)]


@pytest.mark.parametrize("fp32", [0, 1])
@pytest.mark.parametrize("H,D,V,R", LATENT)
def test_latent_attention(nat, H, D, V, R, fp32):
    """Prompts, portions and decode rows; slots used again; several sequences together. The portion sizes put positions on both
    sides of the kernels' token tiles (64, 128) and of the switch between their forms."""
    t = Latent(nat, H, D, V, R, fp32, seed=H + R)
    rng = np.random.default_rng(1)
    T = 330
    q, c = rng.standard_normal((2, T, H * D)).astype(np.float32), rng.standard_normal((2, T, R)).astype(np.float32)
    want = [t.oracle(q[s], c[s]) for s in (0, 1)]
    tol = 3e-5 if fp32 else 3e-3
    for plan in ([[(0, 330)]], [[(0, 64)], [(0, 1)], [(0, 63)], [(0, 1)], [(0, 2)], [(0, 199)]],
                 [[(0, 130), (1, 1)], [(1, 1), (0, 128)], [(0, 1), (1, 1)], [(0, 2), (1, 65), (0, 0)], [(1, 200), (0, 1)], [(1, 1)] ]):
        at = [0, 0]
        for step in plan:
            segs = [(s, at[s], n) for s, n in step if n]
            got = t.run(segs, np.concatenate([q[s, p:p + n] for s, p, n in segs]), np.concatenate([c[s, p:p + n] for s, p, n in segs]),
                        max_len=max(p + n for _, p, n in segs))
            close(got, np.concatenate([want[s][p:p + n] for s, p, n in segs]), tol, f"{step} of {plan}")
            for s, n in step:
                at[s] += n
    # without a sink, without the host's copy of the segments and without a known length
    t.sink = None
    t.dev[4] = None
    got = t.run([(0, 0, 300)], q[0, :300], c[0, :300], host=False)
    close(got, t.oracle(q[0, :300], c[0, :300]), tol, "no sink")
    no_status(nat)
    t.close()


@pytest.mark.parametrize("fp32", [0, 1])
@pytest.mark.parametrize("H,D,V,R", [(4, 64, 64, 128), (2, 128, 128, 512), (3, 40, 24, 56)])
def test_latent_attention_finds_one_far_token(nat, H, D, V, R, fp32):
    """One latent stands out for the queries: its value must come back whole from every place in the cache, from the first
    token to the newest one, past tile and chunk edges, and from nowhere before it is there."""
    t = Latent(nat, H, D, V, R, fp32, seed=3, max_len=1400)
    t.sink[:] = 0.0
    t.dev[4] = f32(nat, t.sink)
    rng = np.random.default_rng(2)
    T = 1300
    key = rng.standard_normal(R)
    for place in (0, 1, 63, 64, 127, 128, 511, 512, 1023, 1024, 1290, 1299):
        c = 0.02 * rng.standard_normal((T, R))
        c = (c / np.sqrt(np.mean(c * c, 1, keepdims=True))).astype(np.float32)
        c[place] = key / np.sqrt(np.mean(key * key))
        q = np.zeros((T, H, D))
        for h in range(H):                      # the query whose absorbed form points at the key
            k = t.uk[h * D:(h + 1) * D].astype(np.float64) @ (t.cn * c[place])
            q[:, h] = k * (30.0 / (k @ k) / t.scale)
        q = q.reshape(T, H * D).astype(np.float32)
        want = t.oracle(q, c)
        got = np.concatenate([t.run([(0, 0, 1290)], q[:1290], c[:1290], 1290)] +
                             [t.run([(0, p, 1)], q[p:p + 1], c[p:p + 1], p + 1) for p in range(1290, T)])
        close(got, want, 2e-4 if fp32 else 2e-2, f"token {place}")
        # the last rows again, together: the form of several rows over cached latents
        close(t.run([(0, 1290, T - 1290)], q[1290:], c[1290:], T), want[1290:], 2e-4 if fp32 else 2e-2, f"token {place}, ten rows")
        if place < T - 1:
            value = (t.uv.astype(np.float64) @ (t.cn * c[place]))
            assert np.abs(want[-1] - value).max() < 0.3 * np.abs(value).max()      # it is that token's value that comes back
    t.close()


def test_latent_attention_batch_decode_lengths(nat):
    """40 sequences of very different lengths decode together (captured form: no known length)."""
    t = Latent(nat, 18, 64, 64, 128, 0, slots=90, max_len=700)
    rng = np.random.default_rng(4)
    lens = [1, 2, 63, 64, 65, 127, 128, 129, 300, 640] * 4
    q, c, want = [], [], []
    for s, n in enumerate(lens):
        qq, cc = rng.standard_normal((n, 18 * 64)).astype(np.float32), rng.standard_normal((n, 128)).astype(np.float32)
        if n > 1:
            t.run([(s, 0, n - 1)], qq[:-1], cc[:-1], n)
        want.append(t.oracle(qq, cc)[-1])
        q.append(qq[-1])
        c.append(cc[-1])
    got = t.run([(s, n - 1, 1) for s, n in enumerate(lens)], np.array(q), np.array(c), host=False)
    close(got, np.array(want), 3e-3)
    t.dev[2] = None       # and without the transposed matrix
    got = t.run([(s, n - 1, 1) for s, n in enumerate(lens)], np.array(q), np.array(c), host=False)
    close(got, np.array(want), 3e-3)
    no_status(nat)
    t.close()


def test_latent_attention_rejects(nat):
    t = Latent(nat, 2, 16, 16, 32, 0, slots=3, max_len=8)
    z = np.zeros((1, 32), np.float32)
    got = t.run([(4, 0, 1)], z, z)          # slot 9 of 3: nothing is read or written
    assert (got == 0).all()
    st = np.zeros(1, np.uint32)
    nat.lib.m40llm_context_take_device_status(nat.ctx, st.ctypes.data)
    assert st[0] & 2
    plain = nat.lib.m40llm_kvcache_create_typed(nat.ctx, 8, 3, 1, 32, 16, N.DT_F16)
    rows = Rows(nat, [(0, 0, 1)])
    b = nat.buf(4096).ptr
    call = N.LatentAttention(b, b, b, None, b, None, b, 64, 2, 16, 16, N.DT_BF16, 1e-5, 1.0)
    assert nat.lib.m40llm_attention_latent_async(nat.ctx, plain, C.byref(call), C.byref(rows.c)) == -4
    call.ld = 63
    assert nat.lib.m40llm_attention_latent_async(nat.ctx, t.kv, C.byref(call), C.byref(rows.c)) == -2
    rot = N.RotaryAttention(b, None, None, b, None, b, 4096, 2, 0, 0, 1e-5, 1.0, 1.0)
    assert nat.lib.m40llm_attention_rotary_async(nat.ctx, t.kv, C.byref(rot), C.byref(rows.c)) == -4
    nat.lib.m40llm_kvcache_destroy(plain)
    t.close()


# -------------------------------------------------------------------------------------------------- real-gated recurrence
@pytest.mark.parametrize("exact", [0, 1])
@pytest.mark.parametrize("W,B,taps", [(320, 5, 4), (256, 1, 2), (96, 3, 1), (42, 3, 3), (1024, 2, 4), (576, 4, 6)])
def test_rglru(nat, W, B, taps, exact):
    rng = np.random.default_rng(W + B)
    D = W // B
    w = {"conv": 0.5 * rng.standard_normal((W, taps)), "conv.b": 0.3 * rng.standard_normal(W), "ra.b": rng.standard_normal((B, D)),
         "ri.b": rng.standard_normal((B, D)), "lam": np.concatenate([rng.uniform(-14, -6, W // 2), rng.uniform(-6, 25, W - W // 2)])}
    w = {n: a.astype(np.float32) for n, a in w.items()}
    for n in ("ra", "ri"):
        w[n] = b16(1.5 * rng.standard_normal((B, D, D)) / D ** 0.5)
    T = 210
    packed = {s: rng.standard_normal((T, 2 * W)).astype(np.float32) for s in range(3)}
    zeros = np.zeros(W)
    ow = {n: a.astype(np.float64) for n, a in w.items()} | {
        "y": np.concatenate([np.eye(W), np.zeros((W, W))], 1), "x": np.concatenate([np.zeros((W, W)), np.eye(W)], 1),
        "y.b": zeros, "x.b": zeros, "o": np.eye(W)}
    ref = {s: S.rglru(p, np.zeros(W), np.zeros((taps - 1, W)), ow, {"blocks": B}) for s, p in packed.items()}
    state = nat.lib.m40llm_statecache_create_values(nat.ctx, 6, W * (1 + taps))
    dev = [f32(nat, w["conv"]), f32(nat, w["conv.b"]), bits(nat, w["ra"]), f32(nat, w["ra.b"]), bits(nat, w["ri"]), f32(nat, w["ri.b"]),
           f32(nat, w["lam"])]
    ld = 2 * W + 8
    # the state is 32-bit in both modes; f32 sums and functions leave a few units in the last place per token
    tol = 2e-5
    for plan in ([[(0, 210)]], [[(0, 1)]] * 30 + [[(0, 2)]] * 3, [[(0, 65), (1, 1)], [(0, 1), (1, 1), (2, 1)], [(2, 130), (0, 2)], [(2, 1)]],
                 [[(s, 1) for s in range(3)]] * 5):
        at = [0, 0, 0]
        for step in plan:
            segs = [(s, at[s], n) for s, n in step]
            rows = Rows(nat, segs, mul=2, add=1)
            x = np.zeros((rows.n, ld), np.float32)
            x[:, :2 * W] = np.concatenate([packed[s][p:p + n] for s, p, n in segs])
            out = nat.buf(rows.n * W * 4)
            c = N.RgLru(f32(nat, x), *dev, out.ptr, ld, W, B, taps, N.DT_BF16, exact, 8.0)
            assert nat.lib.m40llm_rglru_async(nat.ctx, state, C.byref(c), C.byref(rows.c)) == 0
            nat.sync(1)
            close(out.download(np.float32, (rows.n, W)), np.concatenate([ref[s][0][p:p + n] for s, p, n in segs]), tol, str(step))
            for s, n in step:
                at[s] += n
        if plan == [[(0, 210)]]:
            got = np.zeros(W * (1 + taps), np.float32)
            assert nat.lib.m40llm_statecache_debug_read_values(nat.ctx, state, 1, got.ctypes.data) == 0
            close(got[:W], ref[0][1], tol, "final state")
    no_status(nat)
    nat.lib.m40llm_statecache_destroy(state)
    nat.free_all()


def test_state_caches_do_not_mix(nat):
    st = nat.lib.m40llm_statecache_create_values(nat.ctx, 2, 64)
    out = np.zeros(64, np.float32)
    assert nat.lib.m40llm_statecache_debug_read(nat.ctx, st, 0, out.ctypes.data) == -3
    assert nat.lib.m40llm_statecache_debug_read_values(nat.ctx, st, 2, out.ctypes.data) == -2
    b = nat.buf(4096).ptr
    rows = Rows(nat, [(0, 0, 1)])
    c = N.RgLru(b, b, b, b, b, b, b, b, b, 64, 32, 2, 2, N.DT_BF16, 0, 8.0)
    assert nat.lib.m40llm_rglru_async(nat.ctx, st, C.byref(c), C.byref(rows.c)) == -3      # 64 values, 96 needed
    nat.lib.m40llm_statecache_destroy(st)
    nat.free_all()


# -------------------------------------------------------------------------------------------------- experts
def run_moe(nat, x, logits, corr, up, down, r, ff, add=None, residual=None, post=None, exact=0, act=N.ACT_GELU_ERF):
    rows, K = x.shape
    out = nat.buf(np.asarray(residual, np.float32) if residual is not None else rows * K * 4)
    g = r.get("groups") or {"count": 0, "keep": 0}
    ld = logits.shape[1] + 3
    z = np.zeros((rows, ld), np.float32)
    z[:, :logits.shape[1]] = logits
    c = N.Moe(f32(nat, x), f32(nat, z), None if corr is None else f32(nat, corr), bits(nat, up), bits(nat, down),
              None if add is None else f32(nat, add), out.ptr if residual is not None else None, out.ptr, post or N.Norm(), rows, K, ff,
              r["experts"], r["identity"], r["top"], g["count"], g["keep"], ld, N.DT_BF16, act, exact, r["scale"])
    rc = nat.lib.m40llm_moe_async(nat.ctx, C.byref(c), 1)
    assert rc == 0, rc
    nat.sync(1)
    got = out.download(np.float32, (rows, K))
    nat.free_all()
    no_status(nat)
    return got


def oracle_moe(x, logits, corr, up, down, r, act=S.gelu_erf):
    ids, wts = S.route(logits, np.zeros(logits.shape[1]) if corr is None else corr, r)
    y = np.zeros(x.shape)
    for t in range(len(x)):
        for e, g in zip(ids[t], wts[t]):
            v = x[t].astype(np.float64)
            y[t] += g * (v if e >= r["experts"] else down[e].astype(np.float64) @ act(up[e].astype(np.float64) @ v))
    return y


MOE = [  # experts, identity, top, groups (count, keep), K, ff
    (10, 2, 3, (3, 2), 192, 64), (16, 0, 1, None, 128, 128), (5, 3, 8, None, 64, 72), (60, 4, 6, (8, 3), 256, 200), (7, 1, 2, (4, 1), 54, 19),
    (130, 14, 4, (12, 5), 72, 40), (1, 0, 1, None, 136, 320), (31, 1, 4, (16, 8), 520, 136)]


@pytest.mark.parametrize("rows", [1, 2, 9, 70, 400])
@pytest.mark.parametrize("E,I,top,groups,K,ff", MOE)
def test_experts(nat, rows, E, I, top, groups, K, ff):
    rng = np.random.default_rng(E + rows)
    r = {"experts": E, "identity": I, "top": top, "scale": 1.3}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    x = rng.standard_normal((rows, K)).astype(np.float32)
    logits = (2.0 * rng.standard_normal((rows, E + I))).astype(np.float32)
    if rows > 60:
        logits[:, rng.integers(0, E)] += 3.0          # a crowded expert and, with many of them, empty ones
    corr = (0.3 * rng.standard_normal(E + I) - 0.2).astype(np.float32)      # mostly negative choice scores
    up, down = b16(1.5 * rng.standard_normal((E, ff, K)) / K ** 0.5), b16(rng.standard_normal((E, K, ff)) / ff ** 0.5)
    want = oracle_moe(x, logits, corr, up, down, r)
    for exact in (0, 1):
        got = run_moe(nat, x, logits, corr, up, down, r, ff, exact=exact)
        close(got, want, 1e-5 if exact else 1e-4, f"exact={exact}")
    add, res = rng.standard_normal((rows, K)), rng.standard_normal((rows, K))
    wn = (1 + 0.3 * rng.standard_normal(K)).astype(np.float32)
    got = run_moe(nat, x, logits, None, up, down, r, ff, add=add, residual=res, act=N.ACT_SILU,
                  post=N.Norm(N.NORM_RMS, 1e-4, 0.0, f32(nat, wn), None, 2, 0))
    want = S.group_rms_norm(oracle_moe(x, logits, None, up, down, r, lambda z: z * S.sigmoid(z)) + add, wn, 1e-4, 2) + res
    close(got, want, 2e-4, "shared expert's result, norm, residual")


def test_experts_of_every_kind_of_choice(nat):
    """Hand-made scores: the correction decides who is chosen and not with what weight; only members of the kept group count
    although others score higher; negative choice scores beat excluded ones; identity outputs pass x on."""
    K, ff, E, I = 64, 64, 6, 2
    rng = np.random.default_rng(0)
    x = rng.standard_normal((1, K)).astype(np.float32)
    up, down = b16(rng.standard_normal((E, ff, K)) / 8), b16(rng.standard_normal((E, K, ff)) / 8)
    r = {"experts": E, "identity": I, "top": 2, "scale": 2.0, "groups": {"count": 2, "keep": 1}}
    z = np.log(np.array([[0.05, 0.05, 0.1, 0.2, 0.25, 0.25, 0.05, 0.05]], np.float32))
    for corr, ids in (([0.9, 0, 0, 0, 0, 0, 0, 0], [0, 3]), ([-2] * 4 + [-1, -1.5, -3, -0.9], [4, 7]), ([0] * 6 + [1, 1], [6, 7])):
        corr = np.array(corr, np.float32)
        got_ids, wts = S.route(z, corr, r)
        assert list(got_ids[0]) == ids
        s = np.exp(z[0].astype(np.float64))
        assert np.allclose(wts[0], 2.0 * s[ids] / s[ids].sum(), rtol=1e-5)
        for rows in (1, 3):
            got = run_moe(nat, np.repeat(x, rows, 0), np.repeat(z, rows, 0), corr, up, down, r, ff)
            close(got, np.repeat(oracle_moe(x, z, corr, up, down, r), rows, 0), 1e-4, str(corr))


def test_experts_reject(nat):
    b = nat.buf(65536).ptr
    ok = dict(rows=1, K=64, ff=64, experts=4, identity=0, top=2, groups=2, keep=1, ld_logits=4, w_dtype=N.DT_BF16, act=2, scale=1.0)
    call = lambda **kw: nat.lib.m40llm_moe_async(nat.ctx, C.byref(N.Moe(x=b, logits=b, up=b, down=b, out=b, **{**ok, **kw})), 1)
    assert call(groups=3) == -2 and call(keep=3) == -2 and call(keep=0) == -2 and call(top=3) == -2 and call(ld_logits=3) == -2
    assert call(experts=2000, ld_logits=2000) == -2 and call(act=7) == -3
    assert call(post=N.Norm(N.NORM_POLY, 1e-5, 0.0, b, None)) == -4
    assert nat.lib.m40llm_moe_async(nat.ctx, C.byref(N.Moe()), 1) == -1
    nat.free_all()
