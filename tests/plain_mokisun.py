"""A plain, slow restatement of the Mokisun design in numpy: one function per mechanism, whole sequences at a
time, token by token where the design has a recurrence, no cache and no batching.  It shares nothing with the
engine; the tests compare the engine's logits with it.

A model is (config, weights): `config` is the dictionary of the design's config.json, `weights` maps the
file's tensor names to arrays.  Everything is computed in the arrays' own type (float64 in the tests).

Notation: X is the stack of residual streams [n, streams, width]; a sublayer f with its vectors a (reading), c (writing)
and its matrix M turns it into X'[t] = sum_s M[s, t] X[s] + c[t] (ls * f(norm(sum_s a[s] X[s]))).
"""
import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def tanh_norm(x, W, name):
    """A norm without statistics: a learned squashing of every coordinate."""
    return np.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def rms(v, eps):
    return v / np.sqrt(np.mean(v * v, axis=-1, keepdims=True) + eps)


# ---- attention -----------------------------------------------------------------------------------------------

def rotate_pairs(v, rot):
    """Turns the pairs (2i, 2i + 1) of the first rot.dims values of every head of v [n, heads, size] by p * base^(-2i/dims)."""
    dims = rot["dims"]
    if dims == 0:
        return v
    f = np.asarray(rot["base"], dtype=v.dtype) ** (-2.0 * np.arange(dims // 2) / dims)
    ang = np.arange(v.shape[0], dtype=v.dtype)[:, None] * f[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = v.copy()
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def weights_with_sink(s, sink):
    """Softmax weights of the scores s whose divisor also holds exp(sink)."""
    top = max(s.max(), sink)
    w = np.exp(s - top)
    return w / (w.sum() + np.exp(sink - top))


def head_slopes(H):
    return 2.0 ** (-8.0 * (np.arange(H) + 1.0) / H)


def windowed(q, k, v, scale, size, sinks, slopes):
    """q [n, H, D] over k, v [n, G, .]: the `size` latest keys (the query's own included), an optional slope a head off the scores, a sink
    a head in the divisor."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((n, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(n):
            lo = max(0, i - size + 1)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale
            if slopes is not None:
                s = s - slopes[h] * (i - np.arange(lo, i + 1))
            out[i, h] = weights_with_sink(s, sinks[h]) @ v[lo:i + 1, g]
    return out


def rotary_attention(h, W, p, m, trace=None):
    n = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate_pairs((h @ W[p + "q"].T).reshape(n, H, D), m["rot"])
    k = rotate_pairs((h @ W[p + "k"].T).reshape(n, G, D), m["rot"])
    v = (h @ W[p + "v"].T).reshape(n, G, E)
    o = windowed(q, k, v, m["scale"], m["mask"]["size"], W[p + "sink"], None).reshape(n, H * E)
    if trace is not None:
        trace["attention"] = o
    return o @ W[p + "o"].T


def sloped_attention(h, W, p, m, trace=None):
    """Keys are the values; positions act through a slope a head; the divisor has one added to it."""
    n = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[p + "q"].T).reshape(n, H, D)
    k = (h @ W[p + "k"].T).reshape(n, G, D)
    o = windowed(q, k, k, m["scale"], m["mask"]["size"], np.zeros(H), head_slopes(H)).reshape(n, H * D)
    if trace is not None:
        trace["attention"] = o
    return o @ W[p + "o"].T


# ---- memories with a decay per channel -----------------------------------------------------------------------

def gated_linear(q, k, v, alpha):
    """S = diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t per head; q, k, alpha [n, H, D], v [n, H, E]."""
    n, H, D = q.shape
    o = np.zeros_like(v)
    for h in range(H):
        S = np.zeros((D, v.shape[2]), dtype=v.dtype)
        for t in range(n):
            S = alpha[t, h][:, None] * S + np.outer(k[t, h], v[t, h])
            o[t, h] = S.T @ q[t, h]
    return o


def gla(h, W, p, m, eps, trace=None):
    n = h.shape[0]
    H, D, E = m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).reshape(n, H, D) * D ** -0.5
    k = (h @ W[p + "k"].T).reshape(n, H, D)
    v = (h @ W[p + "v"].T).reshape(n, H, E)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = np.exp(-softplus(-z) / m["tau"]).reshape(n, H, D)
    o = gated_linear(q, k, v, alpha)
    heads = (rms(o, eps) * W[p + "norm"]).reshape(n, H * E) * silu(h @ W[p + "g"].T)
    if trace is not None:
        trace.update(memory=o.reshape(n, H * E), heads=heads)
    return heads @ W[p + "o"].T


def causal_conv(x, taps):
    """x [n, C], taps [C, K]: y[t] = sum_j taps[:, j] x[t - (K - 1) + j], zeros before the start."""
    n, K = x.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((K - 1, x.shape[1]), dtype=x.dtype), x])
    return sum(taps[:, j] * padded[j:j + n] for j in range(K))


def unit(v):
    return v / np.sqrt(np.sum(v * v, axis=-1, keepdims=True) + 1e-6)


def delta_memory(q, k, v, g, beta):
    """S = g_t S; u = beta_t (v_t - S^T k_t); S = S + k_t u^T; o_t = S^T q_t per head; q, k [n, G, D], g [n, H, D], v [n, H, E]."""
    n, H, E = v.shape
    share = H // q.shape[1]
    o = np.zeros_like(v)
    for h in range(H):
        a = h // share
        S = np.zeros((q.shape[2], E), dtype=v.dtype)
        for t in range(n):
            S = g[t, h][:, None] * S
            S = S + np.outer(k[t, a], beta[t, h] * (v[t, h] - S.T @ k[t, a]))
            o[t, h] = S.T @ q[t, a]
    return o


def gated_delta(h, W, p, m, eps, trace=None):
    n = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ W[p + x].T, W[p + x + ".conv"])) for x in ("q", "k", "v"))
    q = unit(q.reshape(n, G, D)) * D ** -0.5
    k = unit(k.reshape(n, G, D))
    v = v.reshape(n, H, E)
    beta = sigmoid(h @ W[p + "b"].T)
    z = ((h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]).reshape(n, H, D)
    g = np.exp(-np.exp(W[p + "A_log"])[None, :, None] * softplus(z))
    o = delta_memory(q, k, v, g, beta)
    gate = sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T)
    heads = (rms(o, eps) * W[p + "norm"]).reshape(n, H * E) * gate
    if trace is not None:
        trace.update(memory=o.reshape(n, H * E), heads=heads)
    return heads @ W[p + "o"].T


def side_by_side(h, W, p, m, eps, trace=None):
    left, right = sloped_attention(h, W, p + "left.", m["left"], trace), gated_delta(h, W, p + "right.", m["right"], eps, trace)
    if trace is not None:
        trace.update(left=left, right=right)
    return m["left_scale"] * left + m["right_scale"] * right


# ---- experts -------------------------------------------------------------------------------------------------

def choose(s, correction, router):
    """The chosen experts of one row of scores s, best first: by s + correction, inside the best groups only."""
    c = s + correction
    groups = router.get("groups")
    if groups:
        size = len(c) // groups["count"]
        best = c.reshape(groups["count"], size).max(axis=1)
        keep = np.argsort(-best, kind="stable")[:groups["keep"]]
        allowed = np.isin(np.arange(len(c)) // size, keep)
        c = np.where(allowed, c, -np.inf)
    return np.argsort(-c, kind="stable")[:router["top"]]


def expert(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def experts_ff(h, W, p, mlp, trace=None):
    router = mlp["router"]
    z = h @ W[p + "router"].T
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s = s / s.sum(axis=1, keepdims=True)
    y = np.zeros_like(h)
    chosen = []
    for t in range(h.shape[0]):
        ids = choose(s[t], W[p + "correction"], router)
        chosen.append(ids)
        for e in ids:
            out = expert(h[t], W, f"{p}e{e}.") if e < router["experts"] else h[t]
            y[t] += router["scale"] * s[t, e] * out
    if trace is not None:
        trace.update(chosen=np.array(chosen), choice=s + W[p + "correction"])
    return y


# ---- a layer and the model -----------------------------------------------------------------------------------

def sublayer(X, W, layer, q, f):
    """One step of the streams through sublayer number q (1 the mixer, 2 the feed-forward)."""
    p = f"{layer}hc{q}."
    u = np.einsum("s,nsw->nw", W[p + "in"], X)
    y = f(tanh_norm(u, W, f"{layer}norm{q}")) * W[f"{layer}ls{q}"]
    return np.einsum("st,nsw->ntw", W[p + "mix"], X) + W[p + "out"][None, :, None] * y[:, None, :]


def layer_forward(X, W, config, i, trace=None):
    l, eps, p = config["layers"][i], config["norm"]["eps"], f"l{i}."
    m, pm = l["mixer"], f"l{i}.mix."
    kinds = {"gla": lambda h: gla(h, W, pm, m, eps, trace), "attention": lambda h: rotary_attention(h, W, pm, m, trace),
             "parallel": lambda h: side_by_side(h, W, pm, m, eps, trace)}
    X = sublayer(X, W, p, 1, kinds[l["type"]])
    if trace is not None:
        trace["mixer"] = X
    if l.get("mlp"):
        X = sublayer(X, W, p, 2, lambda h: experts_ff(h, W, p + "mlp.", l["mlp"], trace))
    return X


def forward(config, W, tokens, traces=None):
    """Logits [n, vocab] of one sequence; `traces` (a list) receives a dictionary per layer with the mechanisms'
    intermediate rows and the streams after the layer under "out"."""
    x = W["embed"][np.asarray(tokens)]
    X = np.repeat(x[:, None, :], config["streams"], axis=1)
    for i in range(len(config["layers"])):
        tr = {} if traces is not None else None
        X = layer_forward(X, W, config, i, tr)
        if traces is not None:
            tr["out"] = X
            traces.append(tr)
    return tanh_norm(X.sum(axis=1), W, "final.norm") @ W["head"].T


def generate_greedy(config, W, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(np.argmax(forward(config, W, tokens)[-1])))
    return tokens[len(prompt):]
