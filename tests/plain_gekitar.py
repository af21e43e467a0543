"""A plain, slow restatement of the Gekitar design in numpy: one function per mechanism, whole sequences at a
time, no cache and no batching.  It shares nothing with the engine; the tests compare the engine's logits with it.

A model is (config, weights): `config` is the dictionary of the design's config.json, `weights` maps the
file's tensor names to arrays.  Everything is computed in the arrays' own type (float64 in the tests).

Notation: x is the residual stream [n, width]; a sublayer reads norm(x) and what it puts out passes a norm of its own
before it joins the stream, x <- x + norm_b(sublayer(norm_a(x))); position p counts from 0.
"""
import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms(v, eps):
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    return v / np.sqrt(np.mean(v * v, axis=-1, keepdims=True) + eps)


def zero_centred_norm(x, w, eps):
    """The blocks' and the model's norm: gains stored around zero."""
    return rms(x, eps) * (1.0 + w)


def embed(config, W, tokens):
    return W["embed"][np.asarray(tokens)] * config["embedding"]["scale"]


# ---- rotation ----------------------------------------------------------------------------------------------

def frequencies(rot):
    """The pairs' frequencies f_i = base^(-2i/dims), and the factor on cosine and sine.  With `scaling` (factor s, original length L, two
    counts of turns, fast and slow): a pair that turns `fast` times or more over L positions keeps f_i, one that turns `slow`
    times or fewer gets f_i / s, those between a blend along a straight line over their numbers."""
    dims, base = rot["dims"], float(rot["base"])
    f = base ** (-2.0 * np.arange(dims // 2) / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def pair_that_turns(times):
        return dims * math.log(sc["original"] / (2.0 * math.pi * times)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_that_turns(sc["fast"])), 0)
    hi = min(math.ceil(pair_that_turns(sc["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(v, positions, rot):
    """Rotates the first rot.dims values of the last axis of v [n, heads, size] in neighbouring pairs; the rest pass."""
    dims = rot["dims"]
    f, factor = frequencies(rot)
    ang = np.asarray(positions, dtype=v.dtype)[:, None] * f.astype(v.dtype)[None, :]
    c, s = (factor * np.cos(ang))[:, None, :], (factor * np.sin(ang))[:, None, :]
    out = v.copy()
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


# ---- mixer: attention with capped scores ---------------------------------------------------------------------

def soft_cap(s, cap):
    return cap * np.tanh(s / cap)


def softmax(s):
    w = np.exp(s - s.max())
    return w / w.sum()


def softmax_with_one(s):
    """Weights when the divisor also holds a one, a key of score 0 without a value."""
    top = max(s.max(), 0.0)
    w = np.exp(s - top)
    return w / (w.sum() + np.exp(-top))


def capped_attention(h, W, p, m, eps, trace=None):
    n = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(n)
    q = (h @ W[p + "q"].T + W[p + "q.b"]).reshape(n, H, D)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).reshape(n, G, D)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).reshape(n, G, E)
    q = rms(rotate(q, pos, m["rot"]), eps)
    k = rms(rotate(k, pos, m["rot"]), eps)
    out = np.zeros((n, H, E), dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        for i in range(n):
            s = soft_cap((k[:i + 1, g] @ q[i, a]) * m["scale"], m["softcap"])
            out[i, a] = softmax_with_one(s) @ v[:i + 1, g]
    if trace is not None:
        trace.update(q=q, k=k, v=v, attention=out.reshape(n, H * E))
    return out.reshape(n, H * E) @ W[p + "o"].T + W[p + "o.b"]


# ---- mixers: attention whose keys and values come from a latent row -------------------------------------------

def latent_rows(h, W, p, m, eps):
    """What a position leaves for later ones: its normed latent, and its rotated key part (shared by the heads)."""
    C = m["kv_rank"]
    down = h @ W[p + "dkv"].T
    c = rms(down[:, :C], eps) * W[p + "dkv.norm"]
    return c, rotate(down[:, None, C:], np.arange(h.shape[0]), m["rot"])[:, 0]


def latent_attention(h, W, p, m, eps, gated, rows, trace=None):
    """`rows`: (latents, shared key parts), this layer's own or another's."""
    n = h.shape[0]
    H, D, E = m["heads"], m["dim"], m["vdim"]
    c, shared_key = rows
    cq = rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (cq @ W[p + "uq"].T).reshape(n, H, D + m["rot_dim"])
    q_plain, q_rot = q[..., :D], rotate(q[..., D:], np.arange(n), m["rot"])
    k_plain = (c @ W[p + "uk"].T).reshape(n, H, D)
    v = (c @ W[p + "uv"].T).reshape(n, H, E)
    size = m["mask"]["size"] if m.get("mask") else n
    out = np.zeros((n, H, E), dtype=h.dtype)
    for a in range(H):
        for i in range(n):
            lo = max(0, i - size + 1)
            s = (k_plain[lo:i + 1, a] @ q_plain[i, a] + shared_key[lo:i + 1] @ q_rot[i, a]) * m["scale"]
            out[i, a] = softmax(s) @ v[lo:i + 1, a]
    heads = out.reshape(n, H * E)
    if gated:
        heads = heads * sigmoid(h @ W[p + "g"].T)
    if trace is not None:
        trace.update(latent=c, shared_key=shared_key, attention=out.reshape(n, H * E), heads=heads)
    return heads @ W[p + "o"].T


# ---- feed-forwards -------------------------------------------------------------------------------------------

def capped_gated_ff(h, W, p, limit):
    g = np.minimum(h @ W[p + "gate"].T, limit)
    u = np.clip(h @ W[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def squared_relu_ff(h, W, p):
    return np.maximum(h @ W[p + "up"].T, 0.0) ** 2 @ W[p + "down"].T


def choose(z, top):
    """Scores over all experts, the `top` largest, their weights."""
    s = softmax(z)
    ids = np.argsort(-s, kind="stable")[:top]
    return ids, s[ids] / (s[ids].sum() + 1e-20)


def routed_ff(h, W, p, mlp, trace=None):
    n, top = h.shape[0], mlp["router"]["top"]
    z = h @ W[p + "router"].T
    y = np.zeros((n, W[p + "e0.down"].shape[0]), dtype=h.dtype)
    chosen = np.zeros((n, top), dtype=np.int64)
    for t in range(n):
        chosen[t], weights = choose(z[t], top)
        for e, w in zip(chosen[t], weights):
            y[t] += w * squared_relu_ff(h[t], W, f"{p}e{int(e)}.")
    if trace is not None:
        trace.update(router=z, chosen=chosen, experts=y.copy())
    if mlp.get("shared"):
        y = y + sigmoid(h @ W[p + "shared.sg"].T) * squared_relu_ff(h, W, p + "shared.")
    return y


# ---- a layer and the model -------------------------------------------------------------------------------------

def layer_forward(x, W, config, i, latents, trace=None):
    """`latents` maps a layer's number to the latent rows it made in this pass."""
    l = config["layers"][i]
    eps, m, p = config["norm"]["eps"], l["mixer"], f"l{i}."
    h = zero_centred_norm(x, W[p + "norm1"], eps)
    if l["type"] == "attention":
        y = capped_attention(h, W, p + "mix.", m, eps, trace)
    elif l["type"] in ("latent_attention", "latent_attention_2"):
        source = m.get("kv_from")
        if source is None:
            latents[i] = latent_rows(h, W, p + "mix.", m, eps)
            source = i
        y = latent_attention(h, W, p + "mix.", m, eps, l["type"] == "latent_attention", latents[source], trace)
    else:
        raise ValueError(l["type"])
    x = x + zero_centred_norm(y, W[p + "norm1b"], eps)
    if trace is not None:
        trace.update(mixer_in=h, mixer_out=y, mixer=x)
    mlp = l.get("mlp")
    if not mlp:
        return x
    h = zero_centred_norm(x, W[p + "norm2"], eps)
    y = capped_gated_ff(h, W, p + "mlp.", mlp["limit"]) if mlp["kind"] == "dense" else routed_ff(h, W, p + "mlp.", mlp, trace)
    if trace is not None:
        trace.update(feed_forward_in=h, feed_forward_out=y)
    return x + zero_centred_norm(y, W[p + "norm2b"], eps)


def forward(config, W, tokens, traces=None):
    """Logits [n, vocab] of one sequence; `traces` (a list) receives a dictionary per layer with the mechanisms'
    intermediate rows and the stream after the layer under "out"."""
    x = embed(config, W, tokens)
    latents = {}
    if traces is not None:
        traces.append({"embed": x})
    for i in range(len(config["layers"])):
        tr = {} if traces is not None else None
        x = layer_forward(x, W, config, i, latents, tr)
        if traces is not None:
            tr["out"] = x
            traces.append(tr)
    return zero_centred_norm(x, W["final.norm"], config["norm"]["eps"]) @ W["head"].T


def generate_greedy(config, W, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(np.argmax(forward(config, W, tokens)[-1])))
    return tokens[len(prompt):]
