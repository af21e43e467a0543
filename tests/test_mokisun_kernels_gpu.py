"""The kernels that came with Mokisun, each by itself against a float64 statement written here: slopes and ones in the divisor in every attention kernel,
the interleaved rotation, the streams between two sublayers, the corrected router, experts without a plan, and the memories with a decay per channel row by
row and in pieces."""
from __future__ import annotations

import math

import numpy as np
import pytest
import torch

from test_kernels_gpu import _paged_case

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def dev():
    return torch.device("cuda:0")


def sloped_reference(refs, n_head, n_kv_head, scale, window, slopes, sink):
    outs = []
    for q, k, v, first in refs:
        Q, L = q.shape[0], k.shape[0]
        o = torch.zeros(Q, n_head, q.shape[2], dtype=torch.float64)
        pos, j = torch.arange(first, first + Q)[:, None], torch.arange(L)[None, :]
        mask = (j <= pos) & ((j > pos - window) if window > 0 else True)
        for h in range(n_head):
            s = (q[:, h] @ k[:, h * n_kv_head // n_head].t()) * scale - slopes[h] * (pos - j)
            e = torch.where(mask, torch.exp(s), torch.zeros(()).double())
            o[:, h] = (e @ v[:, h * n_kv_head // n_head]) / (e.sum(1, keepdim=True) + math.exp(sink))
        outs.append(o.reshape(Q, -1))
    return torch.cat(outs)


def slopes_of(n_head, dev):
    s = [2.0 ** (-8.0 * (h + 1) / n_head) for h in range(n_head)]
    return torch.tensor(s + [-1.0] * n_head, device=dev), s


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n_head,n_kv_head,head_dim,page_size,window", [(4, 4, 16, 16, 0), (6, 2, 48, 32, 90), (5, 1, 64, 64, 70), (4, 2, 24, 16, 33), (12, 3, 128, 16, 88)])
def test_generic_attention_with_slopes(dev, dtype, n_head, n_kv_head, head_dim, page_size, window):
    from liyab_b200 import ops
    scale = 0.9 / math.sqrt(head_dim)
    q, cache, tok_seq, positions, table, refs = _paged_case(dev, dtype, n_head, n_kv_head, head_dim, page_size, [1, 37, 130, 64, 300], [1, 37, 2, 1, 45], seed=head_dim)
    d, slopes = slopes_of(n_head, dev)
    ref = sloped_reference(refs, n_head, n_kv_head, scale, window, slopes, 0.0)
    assert (ref - sloped_reference(refs, n_head, n_kv_head, scale, window, [0.0] * n_head, 0.0)).abs().max() > 0.05
    out = torch.empty_like(q)
    ops.paged_attention_generic(q, cache, tok_seq, positions, table, out, q.shape[0], n_head, n_kv_head, head_dim, page_size, scale, window, distance=d,
                                sink=torch.zeros(n_head, device=dev))
    assert (out.double().cpu() - ref).abs().max().item() < (2e-5 if dtype == torch.float32 else 1.5e-2)


@pytest.mark.parametrize("n_head,n_kv_head,head_dim,page_size,window,splits", [(12, 12, 64, 16, 0, 5), (4, 4, 16, 16, 40, 3), (12, 3, 128, 16, 88, 4), (16, 2, 64, 64, 0, 7),
                                                                               (6, 3, 64, 16, 33, 1), (5, 5, 128, 32, 70, 2)])
def test_decode_attention_with_slopes(dev, n_head, n_kv_head, head_dim, page_size, window, splits):
    from liyab_b200 import ops
    lens = [1, 2, 17, 64, 65, 300, 1024, 33]
    S, scale = len(lens), 0.9 / math.sqrt(head_dim)
    q, cache, tok_seq, positions, table, refs = _paged_case(dev, torch.bfloat16, n_head, n_kv_head, head_dim, page_size, lens, [1] * S, seed=splits)
    d, slopes = slopes_of(n_head, dev)
    ref = sloped_reference(refs, n_head, n_kv_head, scale, window, slopes, 0.0)
    partial = torch.full((S * n_head * splits * (head_dim + 2),), float("nan"), device=dev)
    counters = torch.zeros(S * n_kv_head, dtype=torch.int32, device=dev)
    kinds = [k for k, takes in zip((False, True), ops.decode_attention_kernels(n_head, n_kv_head, head_dim, page_size)) if takes]
    assert kinds
    for tensor_cores in kinds:
        out = torch.full_like(q, float("nan"))
        ops.decode_attention(q, cache, positions, table, out, partial, counters, S, n_head, n_kv_head, head_dim, page_size, scale, window, splits,
                             tensor_cores=tensor_cores, distance=d, sink=torch.zeros(n_head, device=dev))
        assert (out.double().cpu() - ref).abs().max().item() < 1.5e-2, f"tensor_cores={tensor_cores}"


@pytest.mark.parametrize("n_head,n_kv_head,head_dim,page_size,window", [(12, 12, 64, 16, 0), (4, 4, 16, 16, 0), (12, 3, 128, 16, 88), (2, 1, 64, 32, 7), (6, 3, 64, 64, 75)])
def test_prefill_attention_with_slopes(dev, n_head, n_kv_head, head_dim, page_size, window):
    from liyab_b200 import ops
    lens, q_lens = [1, 37, 130, 64, 300, 2, 129, 1024], [1, 37, 2, 1, 45, 2, 65, 200]
    scale = 0.9 / math.sqrt(head_dim)
    q, cache, tok_seq, positions, table, refs = _paged_case(dev, torch.bfloat16, n_head, n_kv_head, head_dim, page_size, lens, q_lens, seed=window)
    q_start = torch.tensor(np.concatenate([[0], np.cumsum(q_lens)]), dtype=torch.int32, device=dev)
    n_past = torch.tensor([l - ql for l, ql in zip(lens, q_lens)], dtype=torch.int32, device=dev)
    d, slopes = slopes_of(n_head, dev)
    ref = sloped_reference(refs, n_head, n_kv_head, scale, window, slopes, 0.0)
    for tcgen05 in [False] + ([True] if ops.prefill_attention_tc_supports(n_head, n_kv_head, head_dim, page_size) else []):
        out = torch.full_like(q, float("nan"))
        ops.prefill_attention(q, cache, q_start, n_past, table, out, len(lens), max(q_lens), n_head, n_kv_head, head_dim, page_size, scale, window, tcgen05=tcgen05,
                              distance=d, sink=torch.zeros(n_head, device=dev))
        assert (out.double().cpu() - ref).abs().max().item() < 1.5e-2, f"tcgen05={tcgen05}"


def test_rotation_of_neighbouring_pairs(dev):
    """Queries and keys rotated in pairs (2i, 2i + 1) of part of a head at positions in the thousands, heads padded, keys and values through scrambled slots."""
    from liyab_b200 import ops
    rng = np.random.default_rng(4)
    T, H, G, D, E, P, rot, ps = 11, 4, 2, 12, 10, 16, 8, 16
    proj = torch.from_numpy(rng.standard_normal((T, H * D + G * (D + E)))).float().to(dev)
    pos = torch.tensor([0, 1, 2, 3, 17, 100, 500, 1100, 2500, 4000, 8000], dtype=torch.int32, device=dev)
    slots = torch.tensor(rng.permutation(3 * ps)[:T], dtype=torch.int32)
    slots[4] = -1
    freq = torch.tensor([300.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32, device=dev)
    q = torch.full((T, H * P), float("nan"), device=dev)
    cache = torch.full((3, 2, G, ps, P), float("nan"), device=dev)
    ops.qkv_rotary_store(proj, 0, H * D, H * D + G * D, None, None, q, cache, slots.to(dev), H, G, D, E, P, ps, 0, 1e-6, pos, freq, rot, interleaved=True)
    ang = pos.double().cpu()[:, None] * freq.double().cpu()[None]

    def turned(x, heads):
        x = x.double().cpu().reshape(T, heads, D).clone()
        a, b = x[..., 0:rot:2].clone(), x[..., 1:rot:2].clone()
        x[..., 0:rot:2] = a * ang.cos()[:, None] - b * ang.sin()[:, None]
        x[..., 1:rot:2] = b * ang.cos()[:, None] + a * ang.sin()[:, None]
        return torch.nn.functional.pad(x, (0, P - D))
    assert (q.double().cpu().reshape(T, H, P) - turned(proj[:, :H * D], H)).abs().max() < 2e-3          # angles of thousands of radians in 32 bits
    assert (q.double().cpu().reshape(T, H, P) - turned(proj[:, :H * D], H))[:7].abs().max() < 1e-4
    k, v = turned(proj[:, H * D:H * D + G * D], G), proj[:, H * D + G * D:].double().cpu().reshape(T, G, E)
    for t in range(T):
        if slots[t] >= 0:
            page, off = divmod(int(slots[t]), ps)
            assert (cache[page, 0, :, off].double().cpu() - k[t]).abs().max() < 2e-3 and (cache[page, 1, :, off, :E].double().cpu() - v[t]).abs().max() < 1e-6
            assert cache[page, 1, :, off, E:].abs().max() == 0
    assert int(torch.isfinite(cache[:, 0, 0, :, 0]).sum()) == T - 1       # the negative slot wrote nothing


# ---------------------------------------------------------------- streams

def plain_choice(z, correction, groups, keep, top, softmax, renormalise, scale):
    s = torch.softmax(z, -1) if softmax else torch.sigmoid(z)
    c = s + correction if correction is not None else s.clone()
    n = z.shape[1]
    best = c.reshape(-1, groups, n // groups).max(-1).values
    allowed = torch.zeros_like(best).scatter_(1, best.topk(keep, -1).indices, 1.0).repeat_interleave(n // groups, -1)
    ids = c.masked_fill(allowed == 0, float("-inf")).topk(top, -1).indices
    w = s.gather(1, ids)
    return ids, scale * (w / w.sum(-1, keepdim=True) if renormalise else w)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("S,W,top", [(1, 64, 2), (2, 96, 3), (3, 50, 2), (4, 128, 1), (5, 36, 4), (9, 33, 2), (2, 2052, 2)])
def test_streams_between_two_sublayers(dev, dtype, S, W, top):
    """Terms of both kinds (scaled rows; gathered experts' results through a plan's places, with identities), the mixing from old to new streams, the next input
    through the tanh norm, the router on it; the opening from fresh rows; the reading of chosen rows."""
    from liyab_b200 import ops
    rng = np.random.default_rng(S * W)
    T, N, real = 13, 12, 9
    r = lambda *s: torch.from_numpy(rng.standard_normal(s)).float().to(dev)
    x0, y1, y2, pairs = r(T, S * W), r(T, W), r(T, W), r(T * top, W)
    own = r(T, W).to(dtype)
    ids = torch.from_numpy(rng.integers(0, N, (T, top)).astype(np.int32)).to(dev)
    place = torch.from_numpy(rng.permutation(T * top).astype(np.int32)).to(dev)
    wts = r(T, top)
    mix, to, ls, nxt, gain, off, alpha = r(S, S), r(S), r(W), r(S), r(W), r(W), torch.tensor([0.7], device=dev)
    matrix, corr = (r(N, W) * W ** -0.5).to(dtype), r(N) * 0.1
    d = lambda t: t.double().cpu()
    for mapped in (True, False):
        x = x0.clone()
        h = torch.full((T, W), float("nan"), dtype=dtype, device=dev)
        rid = torch.full((T, 3), -1, dtype=torch.int32, device=dev)
        rw = torch.full((T, 3), float("nan"), device=dev)
        terms = ops.output_terms([y1, y2], [0.5, -1.5], pairs, place if mapped else None, ids, wts, real, own)
        router = ops.router_args(matrix, 3, rid, rw, correction=corr, groups=4, keep=2, scale=2.5)
        ops.streams_join(x, S, T, terms, mix, to, ls, next_in=nxt, norm=(alpha, gain, off), h=h, router=router)
        y = 0.5 * d(y1) - 1.5 * d(y2)
        for t in range(T):
            for k in range(top):
                p = t * top + k
                row = d(pairs)[int(place.flatten()[p]) if mapped else p] if int(ids[t, k]) < real else d(own)[t]
                y[t] += float(wts[t, k]) * row
        y = y * d(ls)
        X = d(x0).reshape(T, S, W)
        want = torch.einsum("st,nsw->ntw", d(mix), X) + d(to)[None, :, None] * y[:, None]
        assert (d(x).reshape(T, S, W) - want).abs().max() < 2e-5 * max(1.0, want.abs().max())
        hw = torch.tanh(0.7 * torch.einsum("s,nsw->nw", d(nxt), want)) * d(gain) + d(off)
        assert (d(h) - hw).abs().max() < (2e-5 if dtype == torch.float32 else 2e-2)
        z = d(h) @ d(matrix).t()
        wid, ww = plain_choice(z, d(corr), 4, 2, 3, True, False, 2.5)
        assert (rid.cpu() == wid).float().mean() > 0.99 and (d(rw) - ww).abs().max() < 1e-4
    # Opening: every stream equals the fresh row, the first input is made in the same launch.
    x = torch.full((T, S * W), float("nan"), device=dev)
    h = torch.empty(T, W, dtype=dtype, device=dev)
    ops.streams_join(x, S, T, fresh=y1, next_in=nxt, norm=(alpha, gain, off), h=h)
    assert (x.reshape(T, S, W) - y1[:, None]).abs().max() == 0
    assert (d(h) - (torch.tanh(0.7 * d(nxt).sum() * d(y1)) * d(gain) + d(off))).abs().max() < (2e-5 if dtype == torch.float32 else 2e-2)
    # Reading: chosen rows' sums, with and without the norm; nothing is written back.
    rows = torch.tensor([7, 0, 12], dtype=torch.int32, device=dev)
    x, h = x0.clone(), torch.empty(3, W, device=dev)
    ops.streams_join(x, S, 3, rows=rows, h=h)
    assert (d(h) - d(x0).reshape(T, S, W).sum(1)[[7, 0, 12]]).abs().max() < 1e-5 and torch.equal(x, x0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("N,W,top,groups,keep,softmax,renormalise", [(22, 96, 3, 2, 1, True, False), (6, 50, 3, 3, 2, True, True), (64, 768, 8, 8, 4, True, False),
                                                                     (1, 32, 1, 1, 1, True, False), (160, 132, 6, 5, 3, False, True), (33, 64, 4, 1, 1, False, False)])
def test_router_with_corrections_and_groups(dev, dtype, N, W, top, groups, keep, softmax, renormalise):
    from liyab_b200 import ops
    rng = np.random.default_rng(N)
    T = 40
    h = torch.from_numpy(rng.standard_normal((T, W))).to(dtype).to(dev)
    m = torch.from_numpy(rng.standard_normal((N, W)) * 2 * W ** -0.5).to(dtype).to(dev)
    corr = torch.from_numpy(rng.uniform(-1.2, -1.0, N)).float().to(dev)         # every choice score is negative
    ids, w = torch.empty(T, top, dtype=torch.int32, device=dev), torch.empty(T, top, device=dev)
    ops.router_choice(ops.router_args(m, top, ids, w, correction=corr, groups=groups, keep=keep, softmax=softmax, renormalise=renormalise, scale=1.5), h)
    wid, ww = plain_choice(h.double().cpu() @ m.double().cpu().t(), corr.double().cpu(), groups, keep, top, softmax, renormalise, 1.5)
    assert torch.equal(ids.cpu().long(), wid) and (w.double().cpu() - ww).abs().max() < 1e-5
    if N > top * 4:
        same = torch.zeros(1, W, dtype=dtype, device=dev)                       # all scores equal: the lowest indices
        ops.router_choice(ops.router_args(m, top, ids[:1], w[:1]), same)
        assert ids[0].tolist() == list(range(top))


@pytest.mark.parametrize("T,top,E,W,F", [(1, 2, 5, 64, 24), (8, 3, 6, 96, 40), (32, 2, 14, 328, 88), (13, 4, 3, 776, 8)])
def test_experts_without_a_plan(dev, T, top, E, W, F):
    from liyab_b200 import ops
    rng = np.random.default_rng(T)
    r = lambda *s: torch.from_numpy(rng.standard_normal(s)).to(torch.bfloat16).to(dev)
    h, gu, down = r(T, W), r(E, 2 * F, W) * W ** -0.5, r(E, W, F) * F ** -0.5
    ids = torch.from_numpy(rng.integers(0, E + 2, (T, top)).astype(np.int32)).to(dev)
    out = ops.experts_direct(h, gu, down, ids).double().cpu()
    for p in range(T * top):
        e = int(ids.flatten()[p])
        if e >= E:
            assert torch.isnan(out[p]).all()                                    # an identity: nobody touched its place
            continue
        a = gu[e].double().cpu() @ h[p // top].double().cpu()
        want = down[e].double().cpu() @ (torch.nn.functional.silu(a[:F]) * a[F:])
        assert (out[p] - want).abs().max() < 3e-2 * max(1.0, want.abs().max())


# ---------------------------------------------------------------- memories with a decay per channel

def memory_case(rng, dev, dtype, H, G, D, E, delta, taps, rank, gate_rank, strong, lens, past):
    """Two halves of work for requests in scrambled slots: `past` rows of each first, then the rest.  Returns the arguments and the float64 reference."""
    t = lambda *s: torch.from_numpy(rng.standard_normal(s)).float().to(dev)
    cols = 2 * G * D + H * E + rank + (gate_rank or H * E) + (H if delta else 0)
    m = dict(n_head=H, kv_head=G, dim=D, vdim=E, delta=delta, taps=taps, unit=delta, gate="sigmoid" if gate_rank else "silu",
             a2=(t(H * D, rank) * rank ** -0.5).to(dtype), g2=(t(H * E, gate_rank) * gate_rank ** -0.5).to(dtype) if gate_rank else None,
             conv=t(2 * G * D + H * E, taps) * 0.7 if taps else None, z_bias=t(H * D) * 2 + (0.0 if delta else 1.0),
             a_log=torch.linspace(-3.0, 4.0 if strong else 0.5, H, device=dev) if delta else None, tau=0.02 if strong else 8.0, norm=t(E) * 0.2 + 1, q_scale=D ** -0.5,
             eps=1e-5)
    return m, {s: t(n, cols) for s, n in enumerate(lens)}


def plain_memory(m, proj):
    """Token by token in float64: (heads before norm and gate, heads after)."""
    f = {k: (v.double().cpu() if torch.is_tensor(v) else v) for k, v in m.items()}
    p = proj.double().cpu()
    H, G, D, E = m["n_head"], m["kv_head"], m["dim"], m["vdim"]
    C, n = 2 * G * D + H * E, proj.shape[0]
    x = p[:, :C]
    if f["conv"] is not None:
        K = m["taps"]
        padded = torch.cat([torch.zeros(K - 1, C).double(), x])
        x = torch.nn.functional.silu(sum(f["conv"][:, j] * padded[j:j + n] for j in range(K)))
    q, k, v = x[:, :G * D].reshape(n, G, D), x[:, G * D:2 * G * D].reshape(n, G, D), x[:, 2 * G * D:].reshape(n, H, E)
    if m["unit"]:
        q, k = (z / torch.sqrt((z * z).sum(-1, keepdim=True) + 1e-6) for z in (q, k))
    q = q * m["q_scale"]
    rank = m["a2"].shape[1]
    z = (p[:, C:C + rank] @ f["a2"].t() + f["z_bias"]).reshape(n, H, D)
    sp = torch.nn.functional.softplus
    log_a = -torch.exp(f["a_log"])[:, None] * sp(z) if m["delta"] else -sp(-z) / m["tau"]
    g_at = C + rank
    gate = torch.sigmoid(p[:, g_at:g_at + m["g2"].shape[1]] @ f["g2"].t()) if m["g2"] is not None else torch.nn.functional.silu(p[:, g_at:g_at + H * E])
    beta = torch.sigmoid(p[:, -H:]) if m["delta"] else None
    o = torch.zeros(n, H, E).double()
    for h in range(H):
        S, g = torch.zeros(D, E).double(), h // (H // G)
        for t in range(n):
            S = torch.exp(log_a[t, h])[:, None] * S
            u = beta[t, h] * (v[t, h] - S.t() @ k[t, g]) if m["delta"] else v[t, h]
            S = S + torch.outer(k[t, g], u)
            o[t, h] = S.t() @ q[t, g]
    heads = o / torch.sqrt((o * o).mean(-1, keepdim=True) + m["eps"]) * f["norm"]
    return o.reshape(n, -1), heads.reshape(n, -1) * gate


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("H,G,D,E,delta,taps,rank,gate_rank", [
    (3, 3, 12, 20, False, 0, 5, 0), (2, 2, 64, 64, False, 0, 16, 0), (1, 1, 33, 5, False, 0, 3, 0), (2, 2, 128, 256, False, 0, 40, 0), (2, 1, 16, 8, False, 2, 4, 6),
    (4, 2, 10, 14, True, 3, 5, 7), (4, 4, 64, 64, True, 4, 24, 24), (5, 1, 7, 33, True, 6, 33, 40), (1, 1, 1, 1, True, 1, 1, 1), (2, 1, 128, 128, True, 4, 16, 16),
    (2, 2, 256, 100, True, 2, 8, 8)])
def test_channel_memory(dev, dtype, strong, H, G, D, E, delta, taps, rank, gate_rank):
    """Every way of cutting: row by row (decode steps with the ring's own write, short portions), in pieces, one after the other over the same state, requests of unequal
    length in scrambled slots; decays so strong that a piece's sums reach hundreds."""
    from liyab_b200 import ops
    rng = np.random.default_rng(D * E + taps)
    lens = [70, 5, 33, 1, 97]
    m, proj = memory_case(rng, dev, dtype, H, G, D, E, delta, taps, rank, gate_rank, strong, lens, None)
    want = {s: plain_memory(m, p) for s, p in proj.items()}
    slots_of = [3, 0, 5, 1, 2]
    floats = H * D * E + taps * (2 * G * D + H * E) + 5
    tol = dict(o=(4e-5 if not strong else 2e-4), heads=3e-4 if dtype == torch.float32 else 2e-2)
    # cuts: per step, how many rows every request brings (0: it sits the step out)
    plans = {"pieces": [lens], "halves": [[40, 2, 31, 1, 50], [30, 3, 2, 0, 47]], "rows": [[2, 1, 2, 1, 3], [1, 1, 1, 0, 1], [1, 1, 1, 0, 1], [66, 2, 29, 0, 92]],
             "decode": [[33, 2, 16, 0, 64]] + [[1, 1, 1, 1, 1]] + [[1, 1, 1, 0, 1]] * 2}
    for kind, steps in plans.items():
        state = torch.zeros(6, floats, device=dev)
        at = [0] * len(lens)
        for counts in steps:
            live = [s for s, c in enumerate(counts) if c > 0]
            rows = torch.cat([proj[s][at[s]:at[s] + counts[s]] for s in live])
            T, HE = rows.shape[0], H * E
            i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
            positions = i32([at[s] + i for s in live for i in range(counts[s])])
            tok_seq = i32([i for i, s in enumerate(live) for _ in range(counts[s])])
            q_start = i32(np.concatenate([[0], np.cumsum([counts[s] for s in live])]).tolist())
            o, heads = torch.full((T, HE), float("nan"), device=dev), torch.full((T, HE), float("nan"), dtype=dtype, device=dev)
            longest = max(counts)
            ops.channel_memory(m, rows.contiguous(), positions, tok_seq, q_start, i32([slots_of[s] for s in live]), state, heads, o, pieces=longest >= 16,
                               decode_only=longest == 1)
            lo = 0
            for s in live:
                n = counts[s]
                wo, wh = (w[at[s]:at[s] + n] for w in want[s])
                err = (o[lo:lo + n].double().cpu() - wo).abs().max() / max(want[s][0].abs().max(), 1e-6)
                assert err < tol["o"], (kind, s, at[s], float(err))
                if E > 1:                                                       # a norm over one value is its sign
                    bad = (heads[lo:lo + n].double().cpu() - wh).abs()
                    scale = 1 + (1 / torch.sqrt((wo.reshape(n, H, E) ** 2).mean(-1) + m["eps"]) * want[s][0].abs().max()).repeat_interleave(E, 1)
                    assert (bad / scale).max() < tol["heads"], (kind, s, at[s])
                at[s] += n
                lo += n
        assert state[4].abs().max() == 0                                        # a slot that nobody holds


@pytest.mark.parametrize("E", [1, 3, 16, 64, 256, 300])
@pytest.mark.parametrize("n_pairs", [1, 31, 256, 257, 1000, 4096, 5003])
def test_expert_plan(dev, n_pairs, E):
    """Pairs sorted by expert, stably, whichever kernel makes the plan; pairs whose expert has no matrix stand nowhere in it."""
    from liyab_b200 import ops
    ids = torch.from_numpy(np.random.default_rng(n_pairs).integers(0, E + 2, n_pairs).astype(np.int32))
    offsets, place, pair_at = ops.expert_plan(ids.to(dev), E)
    real = [p for p in range(n_pairs) if ids[p] < E]
    order = sorted(real, key=lambda p: int(ids[p]))
    assert offsets.tolist() == [sum(int(ids[p]) < e for p in real) for e in range(E)] + [len(real)]
    assert pair_at[:len(real)].tolist() == order and place[order].tolist() == list(range(len(real)))
    assert bool((pair_at[len(real):] == -7).all()) and bool((place[[p for p in range(n_pairs) if ids[p] >= E]] == -7).all())
