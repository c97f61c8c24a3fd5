"""Lamutar: gated rotary-value attention and generalised-delta-rule layers, dynamic-tanh norms before and after every
sublayer, and an optional block of layers that runs several times on the same weights.

This file only reads the configuration and names the tensors; the mechanisms are the framework's (host.StackModel,
m40llm_linear / _attention_rotary / _delta_rule).
"""
from __future__ import annotations

import math

from .. import host, native
from . import register
from .stack import StackWeights, rotary_tables

DECAY_SCALE = -math.exp(-0.5)   # log decay = DECAY_SCALE * sigmoid(...)
UNIT_EPS = 1e-6                 # inside the root of the unit key


@register("Lamutar")
class LamutarSpec:
    def __init__(self, config: dict):
        self.config = config
        self.width, self.vocab = int(config["width"]), int(config["vocab"])
        self.eps = float(config["norm"]["eps"])
        self.soft_cap = float(config.get("logit_softcap") or 0.0)
        self.layers = config["layers"]
        self.loop = config.get("loop")
        for i, layer in enumerate(self.layers):
            if layer["type"] not in ("attention", "general_delta"):
                raise ValueError(f"layer {i}: unknown type {layer['type']!r}")
            if layer.get("mlp") and layer["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {layer['mlp']['kind']!r}")
        if self.loop and not (0 <= self.loop["start"] < self.loop["stop"] <= len(self.layers) and self.loop["times"] >= 1):
            raise ValueError(f"loop {self.loop} does not fit {len(self.layers)} layers")

    def order(self) -> list[tuple[str, int]]:
        """What runs, in order: ("layer", index) and ("join", number of the pass)."""
        n = len(self.layers)
        if not self.loop:
            return [("layer", i) for i in range(n)]
        start, stop = self.loop["start"], self.loop["stop"]
        runs = [("layer", i) for i in range(start)]
        for t in range(self.loop["times"]):
            runs += [("join", t)] + [("layer", i) for i in range(start, stop)]
        return runs + [("layer", i) for i in range(stop, n)]

    def build(self, nat, tensors, dtype: str = "bfloat16", sequences: int = 8, max_len: int = 4096,
              max_rows: int = 2048) -> host.StackModel:
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {dtype!r}")
        w = tensors if isinstance(tensors, StackWeights) else StackWeights(nat, tensors)
        W, V = self.width, self.vocab
        cfg = host.StackCfg(hidden=W, vocab=V, w_dtype=native.DT_BF16, exact=1 if dtype == "float32" else 0,
                            sequences=sequences, max_len=max_len, max_rows=max_rows, soft_cap=self.soft_cap,
                            embeddings=w.matrix("embed", shapes=[(V, W)]), lm_head=w.matrix("head", shapes=[(V, W)]),
                            norm=w.dynamic_tanh("final.norm", W))
        descs: dict[int, host.StackLayerDesc] = {}
        runs = []
        for what, i in self.order():
            if what == "join":
                runs.append((w.matrix("loop.in", shapes=[(W, 2 * W)]), w.vector("loop.step", W, row=i)))
                continue
            if i not in descs:
                descs[i] = self._layer(w, i)
            runs.append(descs[i])
        return host.StackModel(nat.ctx, cfg, runs)

    def _layer(self, w: StackWeights, i: int) -> host.StackLayerDesc:
        layer, W, p = self.layers[i], self.width, f"l{i}."
        m, mix = layer["mixer"], f"l{i}.mix."
        d = host.StackLayerDesc(eps=self.eps, norm1=w.dynamic_tanh(p + "norm1", W), norm1b=w.dynamic_tanh(p + "norm1b", W))
        H = int(m["heads"])
        if layer["type"] == "attention":
            G, K, V, rot = int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), m["rot"]
            turns, amp = rotary_tables(rot["base"], int(rot["dims"]), rot.get("scaling"))
            d.mixer = host.MIXER_ROTARY_ATTENTION
            d.w_in = w.matrix(*(mix + n for n in "qkvg"), shapes=[(H * K, W), (G * K, W), (G * V, W), (H, W)])
            d.n_in = H * K + G * (K + V) + H
            d.w_out = w.matrix(mix + "o", shapes=[(W, H * V)])
            d.q_heads, d.kv_heads, d.k_dim, d.v_dim, d.has_gate = H, G, K, V, 1
            d.q_norm, d.k_norm = w.vector(mix + "q.norm", H * K), w.vector(mix + "k.norm", G * K)
            d.k_pairs, d.k_turns, d.k_amp, d.scale = len(turns), w.table(turns), amp, float(m["scale"])
            d.v_turns = w.table(rotary_tables(rot["base"], V, None)[0])   # values turn unscaled over all their dimensions
        else:
            D, R = int(m["dim"]), w.shape(mix + "w1")[0]
            HD = H * D
            d.mixer = host.MIXER_DELTA_RULE
            d.w_in = w.matrix(*(mix + n for n in ("r", "k", "v", "g", "a", "w1")), shapes=[(HD, W)] * 5 + [(R, W)])
            d.n_in = 5 * HD + R
            d.w_out = w.matrix(mix + "o", shapes=[(W, HD)])
            d.heads, d.dim, d.rank = H, D, R
            d.decay_scale, d.unit_eps = DECAY_SCALE, UNIT_EPS
            d.w2 = w.matrix(mix + "w2", shapes=[(HD, R)])
            d.w0, d.a_bias, d.o_norm = (w.vector(mix + n, HD) for n in ("w0", "a.b", "norm"))
        if layer.get("mlp"):
            F, mlp = int(layer["mlp"]["ff"]), p + "mlp."
            d.norm2, d.norm2b = w.dynamic_tanh(p + "norm2", W), w.dynamic_tanh(p + "norm2b", W)
            d.ff, d.act = F, native.ACT_GELU_TANH
            d.gate, d.up = w.matrix(mlp + "gate", shapes=[(F, W)]), w.matrix(mlp + "up", shapes=[(F, W)])
            d.down = w.matrix(mlp + "down", shapes=[(W, F)])
        return d
