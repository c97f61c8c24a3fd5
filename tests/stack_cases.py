"""Random layer-stack models for the tests: small configurations, weights already rounded to bfloat16."""
from __future__ import annotations

import json
import os

import numpy as np

import helpers


def attention(heads, kv_heads, dim, vdim, dims, base=10000.0, scale=None, scaling=None, ff=80):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = scaling
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot,
                      "scale": dim ** -0.5 if scale is None else scale}}


def delta(heads, dim, ff=80):
    return {"type": "general_delta", "mlp": {"kind": "dense", "ff": ff} if ff else None, "mixer": {"heads": heads, "dim": dim}}


def config(layers, width=96, vocab=140, loop=None, cap=20.0, eps=1e-5):
    c = {"architecture": "Lamutar", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        c["loop"] = loop
    if cap:
        c["logit_softcap"] = cap
    return c


def random_weights(cfg, seed, rank=24):
    helpers.load_package()
    from m40_llm_b200.weights import bf16_to_f32, f32_to_bf16
    rng = np.random.default_rng(seed)
    out = {}

    def put(name, a):
        out[name] = bf16_to_f32(f32_to_bf16(np.asarray(a, np.float32)))

    def mat(name, n, k, gain=1.0):
        put(name, rng.standard_normal((n, k)) * gain / np.sqrt(k))

    def norm(name, n):
        put(name, 1.0 + 0.2 * rng.standard_normal(n))
        put(name + ".b", 0.1 * rng.standard_normal(n))
        put(name + ".alpha", rng.uniform(0.4, 1.2))

    width, vocab = cfg["width"], cfg["vocab"]
    put("embed", rng.standard_normal((vocab, width)))
    mat("head", vocab, width, 3.0)
    norm("final.norm", width)
    if cfg.get("loop"):
        mat("loop.in", width, 2 * width)
        put("loop.step", 0.5 * rng.standard_normal((cfg["loop"]["times"], width)))
    for i, ly in enumerate(cfg["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if ly["mlp"] else ()):
            norm(p + n, width)
        H, D = m["heads"], m["dim"]
        if ly["type"] == "attention":
            G, V = m["kv_heads"], m["vdim"]
            mat(p + "mix.q", H * D, width)
            mat(p + "mix.k", G * D, width)
            mat(p + "mix.v", G * V, width, 1.5)
            mat(p + "mix.g", H, width)
            mat(p + "mix.o", width, H * V, 1.5)
            put(p + "mix.q.norm", 1.0 + 0.3 * rng.standard_normal(H * D))
            put(p + "mix.k.norm", 1.0 + 0.3 * rng.standard_normal(G * D))
        else:
            for n in "rkvga":
                mat(p + "mix." + n, H * D, width)
            mat(p + "mix.w1", rank, width)
            mat(p + "mix.w2", H * D, rank, 1.5)
            mat(p + "mix.o", width, H * D, 1.5)
            put(p + "mix.w0", rng.uniform(-6.0, 2.0, H * D))
            put(p + "mix.a.b", rng.standard_normal(H * D))
            put(p + "mix.norm", 1.0 + 0.3 * rng.standard_normal(H * D))
        if ly["mlp"]:
            F = ly["mlp"]["ff"]
            mat(p + "mlp.gate", F, width, 1.5)
            mat(p + "mlp.up", F, width, 1.5)
            mat(p + "mlp.down", width, F, 1.5)
    return out


def write_model(folder, cfg, weights):
    helpers.load_package()
    from m40_llm_b200 import weights as wt
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    wt.write(os.path.join(folder, "model.safetensors"), weights)
    return str(folder)


YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}

CASES = {
    # both head sizes of the tensor-core attention, a loop over a mixed block
    "loop_tiles": config([delta(3, 24), attention(4, 2, 64, 64, 32, scaling=YARN), delta(3, 24, ff=0), attention(2, 2, 128, 128, 64)],
                         loop={"start": 1, "stop": 3, "times": 3}),
    # key and value sizes differ, one key/value head, full rotation, no loop, no feed-forward on one layer, no cap
    "odd_sizes": config([attention(5, 1, 48, 80, 48, base=500.0, ff=0), delta(2, 36), attention(6, 3, 32, 16, 8, base=1e5, scaling=YARN)],
                        width=104, vocab=77, cap=None, eps=1e-3),
    # a single looped layer, a state wider than the residual, width not a multiple of 8 (f32 kernels throughout)
    "unaligned": config([attention(3, 3, 20, 12, 4), delta(2, 70, ff=33)], width=50, vocab=51, cap=5.0,
                        loop={"start": 0, "stop": 2, "times": 1}),
    # recurrent layers only
    "delta_only": config([delta(1, 128), delta(4, 17)], width=128, vocab=300),
}
