"""Random layer-stack models for the tests: small configurations, weights already rounded to bfloat16."""
from __future__ import annotations

import copy
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


# ------------------------------------------------------------------------------------------------------- Sidalorn
def latent(heads, dim, vdim, rank, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank,
                                                              "scale": dim ** -0.5 if scale is None else scale}}


def rglru(width, blocks, conv, mlp=None):
    return {"type": "rglru", "mlp": mlp, "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, identity, top, ff, groups=None, scale=1.0, shared=None):
    r = {"experts": n, "identity": identity, "top": top, "scale": scale}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    spec = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        spec["shared"] = {"ff": shared}
    return spec


def sidalorn(layers, width, vocab, taps, groups=1, eps=1e-5):
    return {"architecture": "Sidalorn", "canon": {"taps": taps}, "layers": layers, "norm": {"eps": eps, "groups": groups},
            "vocab": vocab, "width": width}


def sidalorn_weights(cfg, seed):
    """Random tensors rounded to bfloat16; sinks and corrections are large enough to matter."""
    helpers.load_package()
    from m40_llm_b200.weights import bf16_to_f32, f32_to_bf16
    rng = np.random.default_rng(seed)
    out = {}

    def put(name, a):
        out[name] = bf16_to_f32(f32_to_bf16(np.asarray(a, np.float32)))

    def mat(name, n, k, gain=1.0):
        put(name, rng.standard_normal((n, k)) * gain / np.sqrt(k))

    def near_one(name, *shape):
        put(name, 1.0 + 0.3 * rng.standard_normal(shape))

    W = cfg["width"]
    put("embed", rng.standard_normal((cfg["vocab"], W)))
    mat("head", cfg["vocab"], W, 3.0)
    near_one("final.norm", W)
    for i, ly in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", ly["mixer"], ly["mlp"]
        put(p + "canon1", 0.4 * rng.standard_normal((W, cfg["canon"]["taps"])))
        near_one(p + "norm1", W)
        if ly["type"] == "latent_attention":
            H, D, V, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
            mat(p + "mix.q", H * D, W, 1.5)
            mat(p + "mix.dkv", R, W)
            near_one(p + "mix.dkv.norm", R)
            mat(p + "mix.uk", H * D, R, 1.5)
            mat(p + "mix.uv", H * V, R)
            put(p + "mix.sink", rng.uniform(-1.0, 3.0, H))
            mat(p + "mix.o", W, H * V)
        else:
            D, B = m["width"], m["blocks"]
            for n in "yx":
                mat(p + "mix." + n, D, W, 1.5)
                put(p + f"mix.{n}.b", 0.3 * rng.standard_normal(D))
            put(p + "mix.conv", 0.5 * rng.standard_normal((D, m["conv"])))
            put(p + "mix.conv.b", 0.3 * rng.standard_normal(D))
            for n in ("ra", "ri"):
                put(p + "mix." + n, 1.5 * rng.standard_normal((B, D // B, D // B)) / np.sqrt(D // B))
                put(p + f"mix.{n}.b", rng.standard_normal((B, D // B)))
            put(p + "mix.lam", rng.uniform(-9.0, 0.5, D))
            mat(p + "mix.o", W, D)
        if not mlp:
            continue
        near_one(p + "norm2", W)
        if mlp["kind"] == "dense":
            mat(p + "mlp.up", mlp["ff"], W)
            mat(p + "mlp.down", W, mlp["ff"])
            put(p + "mlp.act", rng.uniform(0.3, 1.0, 4) * rng.choice([-1, 1], 4))
            continue
        r, F = mlp["router"], mlp["expert"]["ff"]
        n = r["experts"] + r["identity"]
        for e in range(r["experts"]):
            mat(p + f"mlp.e{e}.up", F, W, 1.5)
            mat(p + f"mlp.e{e}.down", W, F, 1.5)
        mat(p + "mlp.router", n, W, 1.5)
        put(p + "mlp.correction", 0.3 * rng.standard_normal(n))
        if mlp.get("shared"):
            mat(p + "mlp.shared.up", mlp["shared"]["ff"], W, 1.5)
            mat(p + "mlp.shared.down", W, mlp["shared"]["ff"], 1.5)
    return out


def clear_tokens(oracle, n, rng, margin=0.01):
    """Random tokens at which no choice of experts is a close call, so that 16-bit rounding cannot turn one; `oracle` is a
    SidalornOracle, reset before and after."""
    oracle.reset()
    out = []
    while len(out) < n:
        before = copy.deepcopy(oracle.state)
        t = int(rng.integers(0, oracle.cfg["vocab"]))
        oracle.step([t])
        if oracle.margin[0] >= margin:
            out.append(t)
        else:
            oracle.state = before
    oracle.reset()
    return np.array(out)


SIDALORN = {
    # shapes of the tensor-core kernels; experts, groups and a shared expert; a layer without a feed-forward
    "tiles": sidalorn([latent(6, 64, 64, 128, mlp=experts(10, 2, 3, 64, groups=(3, 2), scale=1.7, shared=96)),
                       rglru(320, 5, 4, mlp=dense(200)), latent(2, 128, 128, 256), rglru(128, 2, 2, mlp=experts(5, 0, 1, 72))],
                      width=192, vocab=210, taps=4, groups=3),
    # more than 16 heads, key and value sizes differ, one filter tap, one block, every output chosen, no correction to speak of
    "wide_heads": sidalorn([latent(20, 32, 48, 80, scale=0.3, mlp=dense(136)), rglru(96, 1, 1, mlp=experts(3, 1, 4, 40, shared=24)),
                            latent(3, 96, 16, 512, mlp=experts(6, 3, 2, 48, groups=(9, 4)))],
                           width=160, vocab=99, taps=1, groups=1, eps=1e-3),
    # nothing is a multiple of 8: the f32 kernels in every mode
    "unaligned": sidalorn([rglru(42, 3, 3, mlp=experts(7, 1, 2, 19, groups=(2, 1), scale=0.5, shared=13)),
                           latent(3, 10, 14, 21, mlp=dense(33))], width=54, vocab=61, taps=7, groups=6),
    # recurrent layers only
    "recurrent": sidalorn([rglru(288, 4, 5, mlp=dense(144)), rglru(64, 8, 6)], width=128, vocab=150, taps=2, groups=8),
}
