"""Sidalorn: a causal input convolution in every layer, latent attention with sinks or a real-gated linear recurrence, and a
PolyNorm feed-forward or a group-limited mixture of experts with identity outputs; grouped RMS norms on the sublayers' outputs.

This file only reads the configuration and names the tensors; the mechanisms are the framework's (host.StackModel,
m40llm_linear / _short_conv / _attention_latent / _rglru / _moe).
"""
from __future__ import annotations

from .. import host, native
from . import register
from .stack import StackWeights

RGLRU_DECAY = 8.0   # log a = -RGLRU_DECAY * r * softplus(lam)
MIXERS = ("latent_attention", "rglru")
ALIGN = 8           # packed projections get a row pitch that is a multiple of this


def _aligned(n: int) -> int:
    return (n + ALIGN - 1) // ALIGN * ALIGN


@register("Sidalorn")
class SidalornSpec:
    def __init__(self, config: dict):
        self.config = config
        self.width, self.vocab = int(config["width"]), int(config["vocab"])
        self.eps, self.groups = float(config["norm"]["eps"]), int(config["norm"].get("groups") or 1)
        self.taps = int(config["canon"]["taps"])
        self.layers = config["layers"]
        if self.width % self.groups:
            raise ValueError(f"{self.groups} norm groups do not divide a width of {self.width}")
        for i, layer in enumerate(self.layers):
            if layer["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown type {layer['type']!r}")
            if layer.get("mlp") and layer["mlp"]["kind"] not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward {layer['mlp']['kind']!r}")

    def build(self, nat, tensors, dtype: str = "bfloat16", sequences: int = 8, max_len: int = 4096,
              max_rows: int = 2048) -> host.StackModel:
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {dtype!r}")
        w = tensors if isinstance(tensors, StackWeights) else StackWeights(nat, tensors)
        W, V = self.width, self.vocab
        cfg = host.StackCfg(hidden=W, vocab=V, w_dtype=native.DT_BF16, exact=1 if dtype == "float32" else 0,
                            sequences=sequences, max_len=max_len, max_rows=max_rows,
                            embeddings=w.matrix("embed", shapes=[(V, W)]), lm_head=w.matrix("head", shapes=[(V, W)]),
                            norm=self._norm(w, "final.norm"))
        return host.StackModel(nat.ctx, cfg, [self._layer(w, i) for i in range(len(self.layers))])

    def _norm(self, w: StackWeights, name: str) -> native.Norm:
        return w.rms(name, self.width, self.eps, self.groups)

    def _layer(self, w: StackWeights, i: int) -> host.StackLayerDesc:
        layer, W, p = self.layers[i], self.width, f"l{i}."
        m, mix = layer["mixer"], f"l{i}.mix."
        d = host.StackLayerDesc(eps=self.eps, norm1b=self._norm(w, p + "norm1"))
        d.conv_taps, d.conv_w = self.taps, w.vector(p + "canon1", W * self.taps)
        if layer["type"] == "latent_attention":
            H, K, V, R = (int(m[n]) for n in ("heads", "dim", "vdim", "kv_rank"))
            d.mixer = host.MIXER_LATENT_ATTENTION
            d.n_in = _aligned(H * K + R)
            d.w_in = w.matrix(mix + "q", mix + "dkv", shapes=[(H * K, W), (R, W)], rows=d.n_in)
            d.w_out = w.matrix(mix + "o", shapes=[(W, H * V)])
            d.q_heads, d.k_dim, d.v_dim, d.rank_kv, d.scale = H, K, V, R, float(m["scale"])
            d.c_norm, d.sink = w.vector(mix + "dkv.norm", R), w.vector(mix + "sink", H)
            d.uk, d.uv = w.matrix(mix + "uk", shapes=[(H * K, R)]), w.matrix(mix + "uv", shapes=[(H * V, R)])
            d.uk_t = w.blocks_transposed(mix + "uk", (H * K, R), H)
        else:
            D, B, T = int(m["width"]), int(m["blocks"]), int(m["conv"])
            if D % B:
                raise ValueError(f"layer {i}: {B} blocks do not divide a recurrence of {D}")
            d.mixer = host.MIXER_RGLRU
            d.n_in = _aligned(2 * D)
            d.w_in = w.matrix(mix + "y", mix + "x", shapes=[(D, W), (D, W)], rows=d.n_in)
            d.in_bias = w.vectors((mix + "y.b", mix + "x.b"), (D, D), d.n_in)
            d.w_out = w.matrix(mix + "o", shapes=[(W, D)])
            d.rg_width, d.rg_blocks, d.rg_taps, d.rg_decay = D, B, T, RGLRU_DECAY
            d.rg_conv, d.rg_conv_b = w.vector(mix + "conv", D * T), w.vector(mix + "conv.b", D)
            d.ra, d.ri = (w.matrix(mix + n, shapes=[(B, D // B, D // B)]) for n in ("ra", "ri"))
            d.ra_b, d.ri_b, d.lam = (w.vector(mix + n, D) for n in ("ra.b", "ri.b", "lam"))
        if layer.get("mlp"):
            self._feed_forward(w, d, layer["mlp"], p)
        return d

    def _feed_forward(self, w: StackWeights, d: host.StackLayerDesc, spec: dict, p: str):
        W, mlp = self.width, p + "mlp."
        d.norm2b = self._norm(w, p + "norm2")
        if spec["kind"] == "dense":
            d.ff = int(spec["ff"])
            d.up, d.down = w.matrix(mlp + "up", shapes=[(d.ff, W)]), w.matrix(mlp + "down", shapes=[(W, d.ff)])
            d.mid = native.Norm(native.NORM_POLY, self.eps, 0.0, w.vector(mlp + "act", 4), None, 0, 0)
            return
        r, E, F = spec["router"], int(spec["router"]["experts"]), int(spec["expert"]["ff"])
        d.ff, d.act = F, native.ACT_GELU_ERF
        d.experts, d.identity, d.top = E, int(r.get("identity") or 0), int(r["top"])
        d.router_scale = float(r["scale"])
        if r.get("groups"):
            d.groups, d.keep = int(r["groups"]["count"]), int(r["groups"]["keep"])
        d.up = w.matrix(*(f"{mlp}e{e}.up" for e in range(E)), shapes=[(F, W)] * E)
        d.down = w.matrix(*(f"{mlp}e{e}.down" for e in range(E)), shapes=[(W, F)] * E)
        d.correction = w.vector(mlp + "correction", E + d.identity)
        names, shapes = [mlp + "router"], [(E + d.identity, W)]
        if spec.get("shared"):
            d.shared_ff = int(spec["shared"]["ff"])
            names.insert(0, mlp + "shared.up")
            shapes.insert(0, (d.shared_ff, W))
            d.shared_down = w.matrix(mlp + "shared.down", shapes=[(W, d.shared_ff)])
        d.n_router = _aligned(sum(s[0] for s in shapes))
        d.w_router = w.matrix(*names, shapes=shapes, rows=d.n_router)
