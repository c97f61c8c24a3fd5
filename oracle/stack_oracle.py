"""Plain, slow float64 statement of the layer-stack mechanisms (numpy), one function per mechanism.

TEST INFRASTRUCTURE ONLY, like oracle.py: the product never imports it and it shares no code with it. Everything works
on one sequence at a time, token rows first: h [T, width]. State that outlives a call (keys, values, the recurrent
matrix) is passed in and out explicitly, so the same functions run a whole prompt, a portion of it or one token.
"""
from __future__ import annotations

import math

import numpy as np
from scipy.special import erf

F = np.float64


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-np.asarray(x, F)))


def gelu_tanh(z):
    z = np.asarray(z, F)
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    x = np.asarray(x, F)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * np.asarray(w, F)


def dyt_norm(x, alpha, w, b):
    """Dynamic tanh: elementwise, no statistics."""
    return np.tanh(float(alpha) * np.asarray(x, F)) * np.asarray(w, F) + np.asarray(b, F)


def rope_freqs(base, dims, scaling=None):
    """(frequencies [dims/2], amplitude). `scaling` = dict(factor, original, fast, slow) switches YaRN on."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], F)
    if not scaling:
        return f, 1.0
    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_half(x, pos, freqs, amp=1.0, sign=1.0):
    """x [T, heads, d]: the pair (m, m + n) of the first 2n = 2 len(freqs) dimensions turns by sign * pos * freqs[m]."""
    n = len(freqs)
    ang = sign * np.asarray(pos, F)[:, None] * freqs[None, :]
    c, s = (np.cos(ang) * amp)[:, None, :], (np.sin(ang) * amp)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * n:]], axis=-1)


def gated_attention(h, pos0, K, V, w, m, eps):
    """w: q k v o g q.norm k.norm; m: heads kv_heads dim vdim scale rot. K [n, G, dim], V [n, G, vdim] hold the earlier
    tokens (keys normalised and turned, values turned). Returns (out [T, width], K, V) with the new rows appended."""
    h = np.asarray(h, F)
    T, H, G, D, VD = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(pos0, pos0 + T)
    q = rms_norm(h @ w["q"].T, w["q.norm"], eps).reshape(T, H, D)
    k = rms_norm(h @ w["k"].T, w["k.norm"], eps).reshape(T, G, D)
    v = (h @ w["v"].T).reshape(T, G, VD)
    f, amp = rope_freqs(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
    fv, _ = rope_freqs(m["rot"]["base"], VD)
    q, k = rotate_half(q, pos, f, amp), rotate_half(k, pos, f, amp)
    v = rotate_half(v, pos, fv)
    K, V = np.concatenate([K, k]), np.concatenate([V, v])
    out = np.zeros((T, H, VD), F)
    for t in range(T):
        n = pos0 + t + 1
        for head in range(H):
            g = head // (H // G)
            s = K[:n, g] @ q[t, head] * m["scale"]
            p = np.exp(s - s.max())
            out[t, head] = (p / p.sum()) @ V[:n, g]
    out = rotate_half(out, pos, fv, sign=-1.0)
    out = out * sigmoid(h @ w["g"].T)[:, :, None]
    return out.reshape(T, H * VD) @ w["o"].T, K, V


def general_delta(h, S, w, m, eps):
    """S [heads, dim (key), dim (value)]; w: r k v g a a.b w0 w1 w2 norm o. Returns (out [T, width], S)."""
    h = np.asarray(h, F)
    T, H, D = len(h), m["heads"], m["dim"]
    shape = (T, H, D)
    r, k, v = ((h @ w[n].T).reshape(shape) for n in ("r", "k", "v"))
    decay = np.exp(-math.exp(-0.5) * sigmoid(np.tanh(h @ w["w1"].T) @ w["w2"].T + w["w0"])).reshape(shape)
    a = sigmoid(h @ w["a"].T + w["a.b"]).reshape(shape)
    u = k / np.sqrt(np.sum(k * k, axis=-1, keepdims=True) + 1e-6)
    S = np.array(S, F)
    o = np.zeros(shape, F)
    for t in range(T):
        for head in range(H):
            old = S[head]
            S[head] = decay[t, head][:, None] * old - np.outer(a[t, head] * u[t, head], u[t, head] @ old) \
                + np.outer(k[t, head], v[t, head])
            o[t, head] = r[t, head] @ S[head]
    o = o / np.sqrt(np.mean(o * o, axis=-1, keepdims=True) + eps)
    y = o.reshape(T, H * D) * w["norm"] * sigmoid(h @ w["g"].T)
    return y @ w["o"].T, S


def gated_mlp(h, gate, up, down, act=gelu_tanh):
    h = np.asarray(h, F)
    return (act(h @ gate.T) * (h @ up.T)) @ down.T


def soft_cap(x, cap):
    return cap * np.tanh(np.asarray(x, F) / cap)


class StackOracle:
    """A whole model: `cfg` as in config.json, `weights` = {tensor name: array}. One sequence, any portions."""

    def __init__(self, cfg, weights):
        self.cfg = cfg
        self.w = {n: np.asarray(a, F) for n, a in weights.items()}
        lp = cfg.get("loop")
        n = len(cfg["layers"])
        self.runs = []  # (layer, pass or None at its first layer)
        if lp:
            self.runs += [(i, None) for i in range(lp["start"])]
            for t in range(lp["times"]):
                self.runs += [(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
            self.runs += [(i, None) for i in range(lp["stop"], n)]
        else:
            self.runs = [(i, None) for i in range(n)]
        self.reset()

    def reset(self):
        self.pos = 0
        self.state = []
        for i, _ in self.runs:
            ly = self.cfg["layers"][i]
            m = ly["mixer"]
            if ly["type"] == "attention":
                self.state.append([np.zeros((0, m["kv_heads"], m["dim"])), np.zeros((0, m["kv_heads"], m["vdim"]))])
            else:
                self.state.append(np.zeros((m["heads"], m["dim"], m["dim"])))

    def norm(self, name, x):
        return dyt_norm(x, self.w[name + ".alpha"], self.w[name], self.w[name + ".b"])

    def step(self, tokens, layer_out=None):
        cfg, eps = self.cfg, self.cfg["norm"]["eps"]
        x0 = self.w["embed"][np.asarray(tokens)]
        x = x0
        for at, (i, t) in enumerate(self.runs):
            ly = cfg["layers"][i]
            if t is not None:
                x = np.concatenate([x, x0], axis=-1) @ self.w["loop.in"].T + self.w["loop.step"][t]
            p = f"l{i}."
            mw = {n[len(p) + 4:]: a for n, a in self.w.items() if n.startswith(p + "mix.")}
            h = self.norm(p + "norm1", x)
            if ly["type"] == "attention":
                y, K, V = gated_attention(h, self.pos, *self.state[at], mw, ly["mixer"], eps)
                self.state[at] = [K, V]
            else:
                y, self.state[at] = general_delta(h, self.state[at], mw, ly["mixer"], eps)
            x = x + self.norm(p + "norm1b", y)
            if ly["mlp"]:
                h = self.norm(p + "norm2", x)
                x = x + self.norm(p + "norm2b", gated_mlp(h, *(self.w[p + "mlp." + n] for n in ("gate", "up", "down"))))
            if layer_out is not None:
                layer_out.append(x)
        self.pos += len(tokens)
        logits = self.norm("final.norm", x) @ self.w["head"].T
        return soft_cap(logits, cfg["logit_softcap"]) if cfg.get("logit_softcap") else logits


# ---------------------------------------------------------------------------------------- Sidalorn's mechanisms
def gelu_erf(z):
    z = np.asarray(z, F)
    return 0.5 * z * (1.0 + erf(z / math.sqrt(2.0)))


def softplus(z):
    return np.logaddexp(0.0, np.asarray(z, F))


def group_rms_norm(x, w, eps, groups):
    """Every one of `groups` consecutive parts of a row is divided by its own root mean square."""
    x = np.asarray(x, F)
    parts = x.reshape(*x.shape[:-1], groups, -1)
    parts = parts / np.sqrt(np.mean(parts * parts, axis=-1, keepdims=True) + eps)
    return parts.reshape(x.shape) * np.asarray(w, F)


def causal_conv(x, past, w, bias=None):
    """x [T, channels], past [taps - 1, channels] the inputs before it, w [channels, taps], the last column being the
    current token's. Returns (out, new past)."""
    taps = w.shape[1]
    seq = np.concatenate([past, np.asarray(x, F)])
    out = np.zeros_like(np.asarray(x, F))
    for t in range(len(out)):
        for j in range(taps):
            out[t] += w[:, j] * seq[t + j]
        if bias is not None:
            out[t] += bias
    return out, seq[len(seq) - (taps - 1):]


def latent_attention(h, C, w, m, eps):
    """w: q dkv dkv.norm uk uv sink o; m: heads dim vdim kv_rank scale. C [n, kv_rank] the earlier tokens' latents.
    Returns (out [T, width], C with the new rows)."""
    h = np.asarray(h, F)
    H, D, V = m["heads"], m["dim"], m["vdim"]
    n0 = len(C)
    C = np.concatenate([C, rms_norm(h @ w["dkv"].T, w["dkv.norm"], eps)])
    q = (h @ w["q"].T).reshape(-1, H, D)
    k, v = (C @ w["uk"].T).reshape(-1, H, D), (C @ w["uv"].T).reshape(-1, H, V)
    out = np.zeros((len(h), H, V), F)
    for t in range(len(h)):
        for head in range(H):
            s = k[:n0 + t + 1, head] @ q[t, head] * m["scale"]
            top = max(s.max(), w["sink"][head])
            p = np.exp(s - top)
            out[t, head] = (p / (p.sum() + np.exp(w["sink"][head] - top))) @ v[:n0 + t + 1, head]
    return out.reshape(len(h), H * V) @ w["o"].T, C


def rglru(h, S, past, w, m):
    """w: y y.b x x.b conv conv.b ra ra.b ri ri.b lam o; S [width] the state, past [taps - 1, width] earlier inputs of the
    convolution. Returns (out [T, model width], S, past)."""
    h = np.asarray(h, F)
    B = m["blocks"]
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u, past = causal_conv(h @ w["x"].T + w["x.b"], past, w["conv"], w["conv.b"])
    parts = u.reshape(len(u), B, -1)
    r = sigmoid(np.einsum("tbi,boi->tbo", parts, w["ra"]) + w["ra.b"]).reshape(u.shape)
    i = sigmoid(np.einsum("tbi,boi->tbo", parts, w["ri"]) + w["ri.b"]).reshape(u.shape)
    a = np.exp(-8.0 * r * softplus(w["lam"]))
    S, out = np.array(S, F), np.zeros_like(u)
    for t in range(len(u)):
        S = a[t] * S + np.sqrt(1.0 - a[t] * a[t]) * i[t] * u[t]
        out[t] = S * y[t]
    return out @ w["o"].T, S, past


def poly_norm(z, coef, eps):
    """a N(z) + b N(z^2) + c N(z^3) + e, N dividing a row by its root mean square."""
    z = np.asarray(z, F)
    n = lambda x: x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    a, b, c, e = coef
    return a * n(z) + b * n(z * z) + c * n(z ** 3) + e


def route(z, correction, r):
    """Router logits z -> chosen experts and their weights per token: (ids [T, top], weights [T, top]).
    r: top scale groups."""
    z = np.asarray(z, F)
    s = np.exp(z - z.max(-1, keepdims=True))
    s /= s.sum(-1, keepdims=True)
    choice = s + correction
    if r.get("groups"):
        parts = choice.reshape(len(z), r["groups"]["count"], -1)
        best = np.argsort(-parts.max(-1), axis=-1, kind="stable")[:, :r["groups"]["keep"]]
        keep = np.zeros(parts.shape[:2], bool)
        np.put_along_axis(keep, best, True, axis=1)
        choice = np.where(keep[:, :, None], parts, -np.inf).reshape(choice.shape)
    ids = np.argsort(-choice, axis=-1, kind="stable")[:, :r["top"]]
    got = np.take_along_axis(s, ids, axis=1)
    return ids, got / (got.sum(-1, keepdims=True) + 1e-20) * r["scale"]


def choice_margin(z, correction, r):
    """Per token, how far the choice is from another one: the smallest gap, in choice scores, between what is taken and what is
    left out, among groups and among outputs."""
    z = np.asarray(z, F)
    s = np.exp(z - z.max(-1, keepdims=True))
    choice = s / s.sum(-1, keepdims=True) + correction
    gaps = np.full(len(z), np.inf)
    if r.get("groups"):
        parts = choice.reshape(len(z), r["groups"]["count"], -1)
        best, keep = np.sort(parts.max(-1), axis=-1)[:, ::-1], r["groups"]["keep"]
        if keep < best.shape[1]:
            gaps = np.minimum(gaps, best[:, keep - 1] - best[:, keep])
        order = np.argsort(-parts.max(-1), axis=-1, kind="stable")[:, :keep]
        choice = np.take_along_axis(parts, order[:, :, None], axis=1).reshape(len(z), -1)
    top = np.sort(choice, axis=-1)[:, ::-1]
    if r["top"] < top.shape[1]:
        gaps = np.minimum(gaps, top[:, r["top"] - 1] - top[:, r["top"]])
    return gaps


def moe(h, w, spec):
    """w: router correction e<i>.up e<i>.down and, with spec["shared"], shared.up shared.down."""
    h = np.asarray(h, F)
    r = spec["router"]
    ids, weights = route(h @ w["router"].T, w["correction"], r)
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, g in zip(ids[t], weights[t]):
            if e >= r["experts"]:
                out[t] += g * h[t]
            else:
                out[t] += g * (w[f"e{e}.down"] @ gelu_erf(w[f"e{e}.up"] @ h[t]))
    if spec.get("shared"):
        out += gelu_erf(h @ w["shared.up"].T) @ w["shared.down"].T
    return out


class SidalornOracle:
    """A whole model, as StackOracle: one sequence, any portions."""

    def __init__(self, cfg, weights):
        self.cfg = cfg
        self.w = {n: np.asarray(a, F) for n, a in weights.items()}
        self.reset()

    def part(self, prefix):
        return {n[len(prefix):]: a for n, a in self.w.items() if n.startswith(prefix)}

    def reset(self):
        taps, width = self.cfg["canon"]["taps"], self.cfg["width"]
        self.state = []
        for ly in self.cfg["layers"]:
            m, st = ly["mixer"], {"canon": np.zeros((taps - 1, width))}
            if ly["type"] == "latent_attention":
                st["C"] = np.zeros((0, m["kv_rank"]))
            else:
                st["S"], st["past"] = np.zeros(m["width"]), np.zeros((m["conv"] - 1, m["width"]))
            self.state.append(st)

    def norm(self, name, x):
        return group_rms_norm(x, self.w[name], self.cfg["norm"]["eps"], self.cfg["norm"]["groups"])

    def step(self, tokens, layer_out=None):
        eps = self.cfg["norm"]["eps"]
        x = self.w["embed"][np.asarray(tokens)]
        self.margin = np.full(len(x), np.inf)   # how clear the experts' choices were, per token of this call
        for i, (ly, st) in enumerate(zip(self.cfg["layers"], self.state)):
            p = f"l{i}."
            mw = self.part(p + "mix.")
            conv, st["canon"] = causal_conv(x, st["canon"], self.w[p + "canon1"])
            if ly["type"] == "latent_attention":
                y, st["C"] = latent_attention(x + conv, st["C"], mw, ly["mixer"], eps)
            else:
                y, st["S"], st["past"] = rglru(x + conv, st["S"], st["past"], mw, ly["mixer"])
            x = x + self.norm(p + "norm1", y)
            if ly["mlp"]:
                fw = self.part(p + "mlp.")
                if ly["mlp"]["kind"] == "dense":
                    y = poly_norm(x @ fw["up"].T, fw["act"], eps) @ fw["down"].T
                else:
                    y = moe(x, fw, ly["mlp"])
                    z = x @ fw["router"].T
                    self.margin = np.minimum(self.margin, choice_margin(z, fw["correction"], ly["mlp"]["router"]))
                x = x + self.norm(p + "norm2", y)
            if layer_out is not None:
                layer_out.append(x)
        return self.norm("final.norm", x) @ self.w["head"].T
