"""Small Gekitar configurations with random weights for the tests, written as model folders.

A differs from layer to layer in every size the design has: grouped and ungrouped key/value heads, query and value sizes that differ, rotations over
part of a head and over all of it, stretched and not, latents of several sizes, windows, a layer that reads another's latent rows through a wider window
and one through a narrower, dense and routed feed-forwards with and without a shared expert, a block without a feed-forward.  B has the sizes the bfloat16
engine's tensor-core kernels take.  C has sizes that fit no kernel's pieces: a width that is no multiple of 8, a window of one position beside one wider
than any prompt, every expert chosen (top = experts), a latent layer first, rotated parts of two values, no rotation at all, a cap far below the
scores, rows shared from a layer without a window.  D keeps sizes equal to one (heads, one expert, heads of one value, a latent of one value).
"""
from __future__ import annotations

import json
import os

import numpy as np


def rotation(dims, base=10000.0, scaling=None):
    r = dict(base=float(base), dims=dims)
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def attention(heads, kv_heads, dim, vdim, scale, cap, rot_dims, base=10000.0, scaling=(3.0, 64, 8.0, 0.5)):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=float(scale), softcap=float(cap), rot=rotation(rot_dims, base, scaling))


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base=10000.0, window=None, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=float(scale), rot=rotation(rot_dim, base))
    if window is not None:
        m["mask"] = dict(size=window)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff, limit):
    return dict(kind="dense", ff=ff, limit=float(limit))


def moe(experts, top, ff, shared=None):
    m = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if shared:
        m["shared"] = dict(ff=shared)
    return m


def layer(mixer, mlp):
    kind = "attention" if "softcap" in mixer else "latent_attention_2" if "mask" in mixer else "latent_attention"
    return dict(type=kind, mixer=mixer, mlp=mlp)


def model(vocab, width, eps, embed_scale, layers):
    return dict(architecture="Gekitar", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=embed_scale), layers=layers)


CONFIG_A = model(160, 96, 1e-5, 3.0, [
    layer(latent(3, 10, 6, 14, 24, 18, 0.25, 300.0, window=20), moe(6, 2, 24, 40)),
    layer(attention(4, 2, 12, 10, 0.9, 4.0, 8, 5000.0), dense(136, 1.0)),
    layer(latent(5, 4, 8, 8, 40, 7, 0.3, 1e4), moe(4, 1, 16, 8)),
    layer(latent(4, 6, 6, 9, 24, 11, 0.3, 300.0, window=33, kv_from=0), None),
    layer(attention(5, 5, 8, 4, 0.7, 30.0, 8, 100.0, None), moe(5, 3, 8)),
    layer(latent(2, 8, 6, 20, 24, 24, 0.2, 300.0, window=7, kv_from=0), dense(48, 2.5)),
    layer(latent(3, 5, 4, 6, 10, 9, 0.4, 50.0), dense(40, 0.5)),
])
CONFIG_B = model(200, 128, 1e-6, 0.5, [
    layer(attention(8, 2, 64, 64, 0.125, 40.0, 32, 5e5, (4.0, 128, 16.0, 1.0)), moe(8, 2, 64, 64)),
    layer(latent(4, 32, 16, 32, 64, 48, 0.14), dense(256, 2.0)),
    layer(latent(16, 16, 32, 16, 128, 80, 0.15, 30000.0, window=40), moe(4, 2, 128, 96)),
    layer(attention(4, 4, 128, 32, 0.09, 1.5, 128, 1e4, None), dense(128, 7.0)),
    layer(latent(8, 48, 32, 64, 128, 64, 0.1, 30000.0, window=48, kv_from=2), dense(192, 3.0)),
])
CONFIG_C = model(97, 100, 1e-4, 1.0, [
    layer(latent(2, 6, 2, 70, 10, 5, 0.4), moe(3, 3, 20, 12)),
    layer(attention(6, 1, 24, 40, 2.0, 2.0, 0, 10000.0, None), dense(50, 1.5)),
    layer(latent(3, 8, 2, 8, 12, 9, 0.35, window=1), None),
    layer(latent(4, 3, 2, 5, 10, 30, 0.5, kv_from=0, window=1000), moe(5, 2, 8)),
    layer(attention(2, 2, 10, 6, 0.4, 50.0, 10, 30.0, (2.0, 32, 3.0, 0.7)), dense(30, 10.0)),
    layer(latent(7, 2, 2, 3, 12, 4, 0.6, kv_from=2, window=19), dense(33, 1.0)),
])
CONFIG_D = model(64, 48, 1e-5, 2.0, [
    layer(attention(1, 1, 2, 1, 1.0, 1.0, 2, 10.0, (2.0, 16, 2.0, 1.0)), moe(1, 1, 8, 1)),
    layer(latent(1, 1, 2, 1, 1, 1, 1.0), dense(1, 1.0)),
    layer(latent(1, 1, 2, 1, 1, 1, 1.0, window=16), moe(2, 1, 1, 4)),
    layer(attention(2, 1, 16, 1, 0.25, 3.0, 16, 1e4), dense(48, 2.0)),
])
CONFIGS = {"A": (CONFIG_A, 51), "B": (CONFIG_B, 52), "C": (CONFIG_C, 53), "D": (CONFIG_D, 54)}


def to_bf16_values(a):
    """Rounds to values that bfloat16 holds, so that the file, the engine in either type and the plain model agree."""
    from liyab_b200.weights import bf16_to_f32, f32_to_bf16
    return bf16_to_f32(f32_to_bf16(np.asarray(a, dtype=np.float32)))


def random_weights(config, seed):
    """The file's tensors, rounded to bfloat16's values."""
    rng = np.random.default_rng(seed)
    V, W = config["vocab"], config["width"]
    out = {}

    def mat(name, rows, cols, std=None):
        out[name] = rng.normal(0.0, std if std is not None else cols ** -0.5, size=(rows, cols))

    def vec(name, n, mean, std):
        out[name] = rng.normal(mean, std, size=n)

    mat("embed", V, W, 1.0)
    mat("head", V, W)
    vec("final.norm", W, 0.0, 0.1)
    for i, l in enumerate(config["layers"]):
        p, m = f"l{i}.", l["mixer"]
        vec(p + "norm1", W, 0.0, 0.2)
        vec(p + "norm1b", W, 0.0, 0.2)
        H, D, E = m["heads"], m["dim"], m["vdim"]
        if l["type"] == "attention":
            G = m["kv_heads"]
            for name, n in (("q", H * D), ("k", G * D), ("v", G * E)):
                mat(p + "mix." + name, n, W)
                vec(p + f"mix.{name}.b", n, 0.0, 0.4)
            vec(p + "mix.o.b", W, 0.0, 0.4)
        else:
            R, C, Q = m["rot_dim"], m["kv_rank"], m["q_rank"]
            mat(p + "mix.dq", Q, W)
            vec(p + "mix.dq.norm", Q, 1.0, 0.2)
            mat(p + "mix.uq", H * (D + R), Q)
            if "kv_from" not in m:
                mat(p + "mix.dkv", C + R, W)
                vec(p + "mix.dkv.norm", C, 1.0, 0.2)
            mat(p + "mix.uk", H * D, C)
            mat(p + "mix.uv", H * E, C)
            if l["type"] == "latent_attention":
                mat(p + "mix.g", H * E, W, 2.0 * W ** -0.5)
        mat(p + "mix.o", W, H * E)
        mlp = l["mlp"]
        if not mlp:
            continue
        vec(p + "norm2", W, 0.0, 0.2)
        vec(p + "norm2b", W, 0.0, 0.2)
        if mlp["kind"] == "dense":
            mat(p + "mlp.gate", mlp["ff"], W)
            mat(p + "mlp.up", mlp["ff"], W)
            mat(p + "mlp.down", W, mlp["ff"])
            continue
        F, X = mlp["expert"]["ff"], mlp["router"]["experts"]
        mat(p + "mlp.router", X, W, 2.0 * W ** -0.5)
        for e in range(X):
            mat(f"{p}mlp.e{e}.up", F, W)
            mat(f"{p}mlp.e{e}.down", W, F)
        if mlp.get("shared"):
            mat(p + "mlp.shared.up", mlp["shared"]["ff"], W)
            mat(p + "mlp.shared.down", W, mlp["shared"]["ff"])
            mat(p + "mlp.shared.sg", 1, W, 2.0 * W ** -0.5)
    return {k: to_bf16_values(v) for k, v in out.items()}


def f64(weights):
    return {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}


def write_model(folder, config, weights):
    from liyab_b200.weights import f32_to_bf16, write_safetensors
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {k: f32_to_bf16(np.asarray(v, dtype=np.float32)) for k, v in weights.items()},
                      tags={k: "BF16" for k in weights})
    return folder


def model_folder(base, name):
    config, seed = CONFIGS[name]
    weights = random_weights(config, seed)
    return write_model(os.path.join(base, f"gekitar_{name}"), config, weights), config, weights
