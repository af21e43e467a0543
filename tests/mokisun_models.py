"""Small Mokisun configurations with random weights for the tests, written as model folders.

A differs from layer to layer in every size the design has: grouped and ungrouped heads, query and value sizes that differ, windows, rotations over part
of a head, convolutions of one and three taps, fast and slow decays, three streams, experts with and without identities and groups, a block without
a feed-forward.  B has the sizes the bfloat16 engine's tensor-core kernels take, four streams and experts in three groups.  C has sizes that fit no
kernel's pieces: a width that is no multiple of 4, five streams, a window of one position beside one wider than any prompt, no rotation, five heads on
one query and key row.  D keeps sizes equal to one (one stream, heads, values, taps, ranks, one expert, one group).
"""
from __future__ import annotations

import json
import os

import numpy as np


def attention(heads, kv_heads, dim, vdim, scale, window, rot_dims, base=10000.0):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=float(scale), mask=dict(size=window),
                                             rot=dict(base=float(base), dims=rot_dims)))


def gla(heads, dim, vdim, tau):
    return dict(type="gla", mixer=dict(heads=heads, dim=dim, vdim=vdim, tau=float(tau)))


def keyed(heads, kv_heads, dim, scale, window):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=float(scale), mask=dict(size=window))


def delta(heads, kv_heads, dim, vdim, conv):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def parallel(left, right, left_scale, right_scale):
    return dict(type="parallel", mixer=dict(left=left, right=right, left_scale=float(left_scale), right_scale=float(right_scale)))


def moe(experts, top, ff, identity=0, groups=1, keep=1, scale=1.0):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, identity=identity, scale=float(scale), groups=dict(count=groups, keep=keep)))


def layer(kind, mlp):
    return dict(kind, mlp=mlp)


def model(vocab, width, streams, eps, layers):
    return dict(architecture="Mokisun", vocab=vocab, width=width, streams=streams, norm=dict(eps=eps), layers=layers)


CONFIG_A = model(150, 96, 3, 1e-5, [
    layer(gla(3, 12, 20, 8.0), moe(6, 2, 24, identity=2, groups=4, keep=2, scale=1.5)),
    layer(attention(4, 2, 12, 10, 0.3, 20, 8, 5000.0), moe(5, 1, 16, identity=1, groups=3, keep=1, scale=2.5)),
    layer(parallel(keyed(4, 2, 12, 0.3, 33), delta(4, 2, 10, 14, 3), 0.7, 1.3), moe(4, 3, 8)),
    layer(attention(5, 5, 8, 4, 0.35, 47, 4, 100.0), None),
    layer(gla(2, 8, 8, 1.0), moe(3, 2, 20, identity=3, groups=2, keep=2, scale=0.5)),
    layer(parallel(keyed(2, 1, 16, 0.25, 9), delta(3, 3, 8, 6, 1), -0.4, 0.9), None),
])
CONFIG_B = model(200, 128, 4, 1e-6, [
    layer(attention(8, 4, 64, 64, 0.125, 48, 16, 20000.0), moe(8, 3, 64, identity=4, groups=3, keep=2, scale=3.0)),
    layer(parallel(keyed(4, 2, 64, 0.12, 80), delta(4, 2, 32, 64, 5), 0.8, 1.1), moe(8, 2, 32)),
    layer(gla(4, 64, 32, 12.0), moe(6, 2, 128, identity=2, groups=2, keep=1, scale=2.0)),
    layer(attention(4, 2, 128, 96, 0.09, 70, 64, 5e5), None),
])
CONFIG_C = model(97, 50, 5, 1e-4, [
    layer(attention(6, 1, 24, 40, 0.2, 1, 0), moe(5, 4, 10, identity=1, groups=3, keep=3, scale=1.2)),
    layer(parallel(keyed(1, 1, 6, 0.5, 1000), delta(5, 1, 7, 33, 6), 1.0, 0.6), moe(7, 2, 9)),
    layer(gla(1, 33, 5, 3.0), None),
    layer(attention(2, 2, 10, 6, 0.4, 1000, 10, 300.0), moe(2, 2, 30, identity=2, groups=4, keep=3, scale=0.8)),
])
CONFIG_D = model(64, 48, 1, 1e-5, [
    layer(gla(1, 1, 1, 5.0), moe(1, 1, 8)),
    layer(parallel(keyed(1, 1, 1, 1.0, 6), delta(1, 1, 1, 1, 1), 1.0, 1.0), moe(1, 1, 1, identity=1, groups=1, keep=1, scale=1.0)),
    layer(attention(1, 1, 2, 1, 1.0, 16, 2, 10.0), moe(2, 2, 4)),
])
CONFIGS = {"A": (CONFIG_A, 61), "B": (CONFIG_B, 62), "C": (CONFIG_C, 63), "D": (CONFIG_D, 64)}
RANKS = {"A": (5, 7), "B": (16, 24), "C": (3, 40), "D": (1, 1)}


def to_bf16_values(a):
    """Rounds to values that bfloat16 holds, so that the file, the engine in either type and the plain model agree."""
    from liyab_b200.weights import bf16_to_f32, f32_to_bf16
    return bf16_to_f32(f32_to_bf16(np.asarray(a, dtype=np.float32)))


def random_weights(config, seed, ranks=(6, 9)):
    """The file's tensors, floats rounded to bfloat16's values.  `ranks`: those of the decays' and of the gates' low-rank maps."""
    rng = np.random.default_rng(seed)
    V, W, S = config["vocab"], config["width"], config["streams"]
    R1, R2 = ranks
    out = {}

    def mat(name, rows, cols, std=None):
        out[name] = rng.normal(0.0, std if std is not None else cols ** -0.5, size=(rows, cols))

    def vec(name, n, mean, std):
        out[name] = rng.normal(mean, std, size=n)

    def norm(name):
        vec(name, W, 1.0, 0.2)
        vec(name + ".b", W, 0.0, 0.2)
        out[name + ".alpha"] = np.asarray(rng.uniform(0.4, 0.9))

    mat("embed", V, W, 1.0)
    mat("head", V, W)
    norm("final.norm")
    for i, l in enumerate(config["layers"]):
        p, m = f"l{i}.", l["mixer"]
        for q in (1, 2) if l["mlp"] else (1,):
            norm(f"{p}norm{q}")
            vec(f"{p}ls{q}", W, 1.0, 0.3)
            vec(f"{p}hc{q}.in", S, 1.0 / S, 0.3 / S ** 0.5)
            vec(f"{p}hc{q}.out", S, 0.8, 0.4)
            out[f"{p}hc{q}.mix"] = np.eye(S) * 0.6 + rng.normal(0.3 / S, 0.2 / S ** 0.5, size=(S, S))
        if l["type"] == "attention":
            H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            mat(p + "mix.q", H * D, W)
            mat(p + "mix.k", G * D, W)
            mat(p + "mix.v", G * E, W)
            vec(p + "mix.sink", H, 0.5, 1.0)
            mat(p + "mix.o", W, H * E)
        elif l["type"] == "gla":
            H, D, E = m["heads"], m["dim"], m["vdim"]
            for x, rows in (("q", H * D), ("k", H * D), ("v", H * E), ("g", H * E)):
                mat(p + "mix." + x, rows, W)
            mat(p + "mix.a1", R1, W)
            mat(p + "mix.a2", H * D, R1)
            vec(p + "mix.a2.b", H * D, 1.5, 2.0)
            vec(p + "mix.norm", E, 1.0, 0.2)
            mat(p + "mix.o", W, H * E)
        else:
            left, right = m["left"], m["right"]
            H, G, D = left["heads"], left["kv_heads"], left["dim"]
            mat(p + "mix.left.q", H * D, W)
            mat(p + "mix.left.k", G * D, W)
            mat(p + "mix.left.o", W, H * D)
            H, G, D, E, K = right["heads"], right["kv_heads"], right["dim"], right["vdim"], right["conv"]
            r = p + "mix.right."
            for x, rows in (("q", G * D), ("k", G * D), ("v", H * E)):
                mat(r + x, rows, W)
                mat(r + x + ".conv", rows, K, 0.8 * K ** -0.5)
                out[r + x + ".conv"][:, -1] += 0.5
            mat(r + "b", H, W)
            out[r + "A_log"] = rng.uniform(-4.0, 1.0, size=H)
            out[r + "dt_bias"] = rng.uniform(-4.0, 0.0, size=H * D)
            vec(r + "norm", E, 1.0, 0.2)
            mat(r + "a1", R1, W)
            mat(r + "a2", H * D, R1)
            mat(r + "g1", R2, W)
            mat(r + "g2", H * E, R2)
            mat(r + "o", W, H * E)
        if l["mlp"]:
            F, router = l["mlp"]["expert"]["ff"], l["mlp"]["router"]
            for e in range(router["experts"]):
                mat(f"{p}mlp.e{e}.gate", F, W)
                mat(f"{p}mlp.e{e}.up", F, W)
                mat(f"{p}mlp.e{e}.down", W, F)
            n = router["experts"] + router["identity"]
            mat(p + "mlp.router", n, W, 2.5 * W ** -0.5)
            # Corrections of either sign, also below every score, that change who is chosen without settling it.
            out[p + "mlp.correction"] = rng.uniform(-1.3, -1.0, size=n)
    return {k: to_bf16_values(v) for k, v in out.items()}


def f64(weights):
    return {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}


def write_model(folder, config, weights):
    from liyab_b200.weights import f32_to_bf16, write_safetensors
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {k: f32_to_bf16(v) for k, v in weights.items()}, tags={k: "BF16" for k in weights})
    return folder


def model_folder(base, name):
    config, seed = CONFIGS[name]
    weights = random_weights(config, seed, RANKS[name])
    return write_model(os.path.join(base, f"mokisun_{name}"), config, weights), config, weights
