"""The kernels that came with Gekitar, each by itself against a float64 statement written here: the soft cap in every attention kernel (32-bit, scalar and
tensor-core decode with split keys, mma.sync and tcgen05 prefill) in both of its forms, queries and keys normed after a rotation with a factor, the launch
between two norms, the router with a gate beside its experts, experts without a gate, and the gate on every value of attention over latent rows."""
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


def capped_attention(refs, n_head, n_kv_head, scale, window, cap, ones):
    """Softmax over cap tanh(s / cap) (cap 0: over s), with one more in the divisor where `ones`."""
    outs, group = [], n_head // n_kv_head
    for q, k, v, first in refs:
        Q, L = q.shape[0], k.shape[0]
        o = torch.zeros(Q, n_head, q.shape[2], dtype=torch.float64)
        pos, j = torch.arange(first, first + Q)[:, None], torch.arange(L)[None, :]
        mask = (j <= pos) & (j > pos - window) if window > 0 else j <= pos
        for h in range(n_head):
            s = (q[:, h] @ k[:, h // group].t()) * scale
            s = cap * torch.tanh(s / cap) if cap > 0 else s
            s = s.masked_fill(~mask, float("-inf"))
            w = torch.exp(s)
            o[:, h] = (w / (w.sum(-1, keepdim=True) + (1.0 if ones else 0.0))) @ v[:, h // group]
        outs.append(o.reshape(Q, -1))
    return torch.cat(outs)


def largest_score(refs, n_head, n_kv_head, scale):
    group = n_head // n_kv_head
    return max(float(((q[:, h] @ k[:, h // group].t()) * scale).abs().max()) for q, k, _, _ in refs for h in range(n_head))


def caps_for(refs, n_head, n_kv_head, scale):
    """(cap, bound) pairs: one deep in the bend, one below the scores' size, and one that is so far above them that the series serves."""
    top = largest_score(refs, n_head, n_kv_head, scale)
    return [(0.3, 0.0), (0.5 * top, 0.0), (4.0 * top, 0.0), (4.0 * top, top)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n_head,n_kv_head,head_dim,page_size,window", [(4, 4, 16, 16, 0), (6, 2, 48, 32, 0), (5, 1, 64, 64, 70), (4, 2, 24, 16, 33), (12, 3, 128, 16, 88),
                                                                        (64, 8, 64, 16, 0)])
def test_soft_cap_in_generic_attention(dev, dtype, n_head, n_kv_head, head_dim, page_size, window):
    from liyab_b200 import ops
    lens, q_lens = [1, 37, 130, 64, 300], [1, 37, 2, 1, 45]
    scale = 2.5 / math.sqrt(head_dim)
    q, cache, tok_seq, positions, table, refs = _paged_case(dev, dtype, n_head, n_kv_head, head_dim, page_size, lens, q_lens, seed=head_dim + n_head)
    ones = torch.zeros(n_head, device=dev)
    plain = capped_attention(refs, n_head, n_kv_head, scale, window, 0.0, True)
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    for cap, _ in caps_for(refs, n_head, n_kv_head, scale):
        ref = capped_attention(refs, n_head, n_kv_head, scale, window, cap, True)
        assert (ref - plain).abs().max() > 5 * tol or cap > largest_score(refs, n_head, n_kv_head, scale), "the cap does not show"
        out = torch.empty_like(q)
        ops.paged_attention_generic(q, cache, tok_seq, positions, table, out, q.shape[0], n_head, n_kv_head, head_dim, page_size, scale, window, sink=ones, soft_cap=cap)
        assert (out.double().cpu() - ref).abs().max().item() < tol, cap
    # A few pairs take the 32-bit kernel arranged around latency: bit for bit the other one's sums.
    if dtype == torch.float32 and n_head == 64:
        few = torch.empty_like(q)
        ops.paged_attention_generic(q[:2], cache, tok_seq[:2], positions[:2], table, few[:2], 2, n_head, n_kv_head, head_dim, page_size, scale, window, sink=ones, soft_cap=cap)
        assert torch.equal(few[:2], out[:2])


@pytest.mark.parametrize("n_head,n_kv_head,head_dim,page_size,window,splits", [
    (12, 12, 64, 16, 0, 1), (12, 12, 64, 16, 0, 5), (4, 4, 16, 16, 0, 3), (12, 3, 128, 16, 88, 4), (16, 2, 64, 64, 0, 7), (4, 4, 32, 16, 5, 16), (2, 1, 256, 16, 200, 9),
    (16, 1, 128, 16, 0, 8), (12, 3, 64, 16, 300, 12)])
def test_soft_cap_in_decode_attention(dev, n_head, n_kv_head, head_dim, page_size, window, splits):
    from liyab_b200 import ops
    lens = [1, 2, 17, 64, 65, 300, 1024, 33]
    S, scale = len(lens), 2.5 / math.sqrt(head_dim)
    q, cache, tok_seq, positions, table, refs = _paged_case(dev, torch.bfloat16, n_head, n_kv_head, head_dim, page_size, lens, [1] * S, seed=7 * head_dim + splits)
    ones = torch.zeros(n_head, device=dev)
    partial = torch.full((S * n_head * splits * (head_dim + 2),), float("nan"), device=dev)
    counters = torch.zeros(S * n_kv_head, dtype=torch.int32, device=dev)
    scalar, tensor = ops.decode_attention_kernels(n_head, n_kv_head, head_dim, page_size)
    for cap, bound in caps_for(refs, n_head, n_kv_head, scale):
        for with_one in (True, False):
            ref = capped_attention(refs, n_head, n_kv_head, scale, window, cap, with_one)
            for tensor_cores in ([False] if scalar else []) + ([True] if tensor else []):
                out = torch.full_like(q, float("nan"))
                ops.decode_attention(q, cache, positions, table, out, partial, counters, S, n_head, n_kv_head, head_dim, page_size, scale, window, splits,
                                     tensor_cores=tensor_cores, sink=ones if with_one else None, soft_cap=cap, score_bound=bound)
                assert (out.double().cpu() - ref).abs().max().item() < 1.5e-2, (tensor_cores, cap, bound)


@pytest.mark.parametrize("n_head,n_kv_head,head_dim,page_size,window", [
    (12, 12, 64, 16, 0), (4, 4, 16, 16, 0), (6, 2, 48, 32, 0), (5, 1, 64, 64, 0), (12, 3, 128, 16, 88), (2, 1, 64, 32, 7), (3, 3, 64, 16, 100)])
def test_soft_cap_in_prefill_attention(dev, n_head, n_kv_head, head_dim, page_size, window):
    """Both tensor-core kernels, portions of every kind in one launch, scores of either sign of the factor."""
    from liyab_b200 import ops
    lens, q_lens = [1, 37, 130, 64, 300, 2, 129, 1024], [1, 37, 2, 1, 45, 2, 65, 200]
    q, cache, tok_seq, positions, table, refs = _paged_case(dev, torch.bfloat16, n_head, n_kv_head, head_dim, page_size, lens, q_lens, seed=head_dim + n_head + window)
    q_start = torch.tensor(np.concatenate([[0], np.cumsum(q_lens)]), dtype=torch.int32, device=dev)
    n_past = torch.tensor([l - ql for l, ql in zip(lens, q_lens)], dtype=torch.int32, device=dev)
    ones = torch.zeros(n_head, device=dev)
    for scale in (2.5 / math.sqrt(head_dim), -1.0 / math.sqrt(head_dim)):
        for cap, bound in caps_for(refs, n_head, n_kv_head, scale):
            ref = capped_attention(refs, n_head, n_kv_head, scale, window, cap, True)
            for tcgen05 in [False] + ([True] if ops.prefill_attention_tc_supports(n_head, n_kv_head, head_dim, page_size) else []):
                out = torch.full_like(q, float("nan"))
                ops.prefill_attention(q, cache, q_start, n_past, table, out, len(lens), max(q_lens), n_head, n_kv_head, head_dim, page_size, scale, window,
                                      tcgen05=tcgen05, sink=ones, soft_cap=cap, score_bound=bound)
                assert ops.device_status() == 0
                assert (out.double().cpu() - ref).abs().max().item() < 1.5e-2, (tcgen05, cap, bound, scale)


def test_a_cap_and_a_penalty_by_distance_are_refused_together(dev):
    from liyab_b200 import ops
    from liyab_b200.status import LiyabError
    q, cache, tok_seq, positions, table, _ = _paged_case(dev, torch.float32, 2, 1, 16, 16, [5], [5], seed=1)
    with pytest.raises(LiyabError, match="soft cap"):
        ops.paged_attention_generic(q, cache, tok_seq, positions, table, torch.empty_like(q), 5, 2, 1, 16, 16, 1.0, distance=torch.zeros(4, device=dev), soft_cap=1.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,E,rot,factor,gains", [(4, 2, 12, 10, 8, 1.3, False), (3, 3, 64, 64, 64, 1.14, False), (2, 1, 128, 40, 96, 0.7, True), (1, 1, 2, 1, 2, 2.0, False),
                                                      (5, 5, 16, 4, 4, 1.5, True), (2, 2, 200, 16, 10, 1.2, False)])
@pytest.mark.parametrize("interleaved", [True, False])
def test_norm_after_a_rotation_with_a_factor(dev, dtype, H, G, D, E, rot, factor, gains, interleaved):
    """Heads over their own root mean square after the rotation, whose cosine and sine carry a factor; far positions, gains, padding, scrambled pages, a slot
    that writes nothing."""
    from liyab_b200 import ops
    rng = np.random.default_rng(H * 100 + D)
    T, page, eps = 23, 16, 1e-2                       # an eps that shows
    P = max(16, 1 << (max(D, E) - 1).bit_length()) if dtype == torch.bfloat16 else (max(D, E) + 3) // 4 * 4
    proj = rng.standard_normal((T, H * D + G * D + G * E + 5)) * 0.5
    qw, kw = rng.uniform(0.5, 1.5, D), rng.uniform(0.5, 1.5, D)
    positions = rng.integers(0, 5000, T)
    freq = 700.0 ** (-2.0 * np.arange(rot // 2) / rot)
    slots = rng.permutation(4 * page)[:T]
    slots[3] = -1

    def rotated_and_normed(x, heads, w):
        x = x.reshape(T, heads, D)
        ang = positions[:, None].astype(np.float64) * freq.astype(np.float32).astype(np.float64)[None, :]
        c, s = factor * np.cos(ang)[:, None, :], factor * np.sin(ang)[:, None, :]
        first, second = (slice(0, rot, 2), slice(1, rot, 2)) if interleaved else (slice(0, rot // 2), slice(rot // 2, rot))
        out = x.copy()
        out[..., first], out[..., second] = x[..., first] * c - x[..., second] * s, x[..., second] * c + x[..., first] * s
        return out / np.sqrt((out * out).mean(-1, keepdims=True) + eps) * (w if gains else 1.0)

    q_ref, k_ref = rotated_and_normed(proj[:, :H * D], H, qw), rotated_and_normed(proj[:, H * D:(H + G) * D], G, kw)
    v_ref = proj[:, (H + G) * D:(H + G) * D + G * E].reshape(T, G, E)
    t = lambda a, ty=torch.float32: torch.tensor(np.asarray(a), dtype=ty, device=dev)
    q_out = torch.full((T, H * P), float("nan"), dtype=dtype, device=dev)
    cache = torch.full((4, 2, G, page, P), float("nan"), dtype=dtype, device=dev)
    ops.qkv_rotary_store(t(proj), 0, H * D, (H + G) * D, t(qw) if gains else None, t(kw) if gains else None, q_out, cache, t(slots, torch.int32), H, G, D, E, P, page, 3, eps,
                         t(positions, torch.int32), t(freq), rot, interleaved=interleaved, rot_factor=factor)
    tol = 3e-4 if dtype == torch.float32 else 2e-2            # angles of thousands of radians in 32-bit
    got = q_out.double().cpu().numpy().reshape(T, H, P)
    assert np.abs(got[..., :D] - q_ref).max() < tol * max(1.0, np.abs(q_ref).max()) and (got[..., D:] == 0).all()
    c = cache.double().cpu().numpy()
    for i in range(T):
        if slots[i] < 0:
            continue
        pg, off = divmod(int(slots[i]), page)
        assert np.abs(c[pg, 0, :, off, :D] - k_ref[i]).max() < tol * max(1.0, np.abs(k_ref).max()) and (c[pg, 0, :, off, D:] == 0).all()
        assert np.abs(c[pg, 1, :, off, :E] - v_ref[i]).max() < tol * max(1.0, np.abs(v_ref).max()) and (c[pg, 1, :, off, E:] == 0).all()
    assert np.isnan(c).sum() == (4 * page - (T - 1)) * 2 * G * P


# ---------------------------------------------------------------- the launch between two norms

def choice(z, top):
    s = torch.softmax(z, dim=-1)
    w, ids = torch.sort(s, dim=-1, descending=True, stable=True)
    w, ids = w[:, :top], ids[:, :top]
    return ids, w / w.sum(-1, keepdim=True)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,T,N,top", [(96, 13, 6, 2), (768, 9, 16, 2), (100, 300, 5, 3), (98, 7, 4, 4), (33, 301, 3, 1), (2052, 5, 40, 6), (200, 310, 4, 2), (512, 300, 4, 1), (768, 301, 4, 2), (1024, 299, 2, 1), (1, 4, 1, 1), (2500, 150, 8, 2), (4100, 310, 2, 1),
                                       (2051, 2, 2, 1), (9000, 3, 2, 1)])
def test_launch_between_two_norms(dev, dtype, W, T, N, top):
    """Terms of both kinds (rows times numbers and times one float a row; routed results through a plan's places and without one), norm, sum into the stream, the next
    input, the router with a gate row on it; without a router; without a next input.  Widths in 16-byte pieces and not, rows for one to sixteen pieces a
    thread, few rows and hundreds (four rows a block)."""
    from liyab_b200 import ops
    rng = np.random.default_rng(W + T)
    r = lambda *s: torch.from_numpy(rng.standard_normal(s)).float().to(dev)
    d = lambda t: t.double().cpu()
    x0, y1, y2, pairs, f2 = r(T, W + 4)[:, :W], r(T, W) * 2, r(T, W), r(T * top, W), r(T)
    ids = torch.from_numpy(rng.integers(0, N, (T, top)).astype(np.int32)).to(dev)
    place = torch.from_numpy(rng.permutation(T * top).astype(np.int32)).to(dev)
    wts, gain, gain2 = r(T, top), r(W) * 0.3, r(W) * 0.3
    matrix = (r(N + 1, W) * 2 * W ** -0.5).to(dtype)
    eps, eps2, scale = 1e-3, 1e-2, 0.7
    rms = lambda v, e: v / torch.sqrt((v * v).mean(-1, keepdim=True) + e)
    for mapped in (True, False):
        y = 0.5 * d(y1) - 1.5 * d(f2)[:, None] * d(y2)
        at = d(place).long() if mapped else torch.arange(T * top)
        y = y + (d(wts)[:, :, None] * d(pairs)[at.reshape(T, top)]).sum(1)
        want = d(x0) + scale * rms(y, eps) * (1.0 + d(gain))
        hw = rms(want, eps2) * (0.5 + d(gain2))
        terms = ops.output_terms([y1, y2], [0.5, -1.5], pairs, place if mapped else None, ids, wts, N, None, factor=(None, f2))
        for mode in ("router", "next", "last"):
            x = torch.empty(T, W + 4, device=dev)[:, :W]
            x.copy_(x0)
            h = torch.full((T, W), float("nan"), dtype=dtype, device=dev) if mode != "last" else None
            rid, rw = torch.full((T, top), -1, dtype=torch.int32, device=dev), torch.full((T, top), float("nan"), device=dev)
            gate = torch.full((T,), float("nan"), device=dev)
            router = ops.router_args(matrix, top, rid, rw, renormalise=True, gate=gate) if mode == "router" else None
            ops.norm_join(x, terms, (gain, 1.0, eps), T, scale, next_norm=(gain2, 0.5, eps2) if h is not None else None, h=h, router=router)
            assert (d(x) - want).abs().max() < 2e-5 * max(1.0, float(want.abs().max())), mode
            if h is None:
                continue
            assert (d(h) - hw).abs().max() < (2e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(hw.abs().max()))
            if router is None:
                continue
            z = d(h) @ d(matrix).t()
            wid, ww = choice(z[:, :N], top)
            assert (rid.cpu() == wid).float().mean() > 0.99
            same = (rid.cpu() == wid).all(1)
            assert (d(rw) - ww)[same].abs().max() < 1e-4 and (d(gate) - torch.sigmoid(z[:, N])).abs().max() < 1e-5
    # A single term (hundreds of rows take a warp a row), with a factor a row.
    for last in (True, False):
        x = torch.empty(T, W + 4, device=dev)[:, :W]
        x.copy_(x0)
        h = None if last else torch.full((T, W), float("nan"), dtype=dtype, device=dev)
        ops.norm_join(x, ops.output_terms([y1], [0.5], factor=(f2,)), (gain, 1.0, eps), T, scale, next_norm=None if last else (gain2, 0.5, eps2), h=h)
        want = d(x0) + scale * rms(0.5 * d(f2)[:, None] * d(y1), eps) * (1.0 + d(gain))
        assert (d(x) - want).abs().max() < 2e-5 * max(1.0, float(want.abs().max()))
        hw = rms(want, eps2) * (0.5 + d(gain2))
        assert last or (d(h) - hw).abs().max() < (2e-5 if dtype == torch.float32 else 1e-2) * max(1.0, float(hw.abs().max()))
    x = torch.empty(T, W + 4, device=dev)[:, :W]
    x.copy_(x0)
    h, gate = torch.full((T, W), float("nan"), dtype=dtype, device=dev), torch.full((T,), float("nan"), device=dev)
    rid, rw = torch.full((T, top), -1, dtype=torch.int32, device=dev), torch.full((T, top), float("nan"), device=dev)
    ops.norm_join(x, ops.output_terms([y1], [0.5], factor=(f2,)), (gain, 1.0, eps), T, scale, next_norm=(gain2, 0.5, eps2), h=h,
                  router=ops.router_args(matrix, top, rid, rw, renormalise=True, gate=gate))
    z = d(h) @ d(matrix).t()
    wid, ww = choice(z[:, :N], top)
    same = (rid.cpu() == wid).all(1)
    assert (d(x) - want).abs().max() < 2e-5 * max(1.0, float(want.abs().max())) and same.float().mean() > 0.99
    assert (d(rw) - ww)[same].abs().max() < 1e-4 and (d(gate) - torch.sigmoid(z[:, N])).abs().max() < 1e-5
    # Without gains: ones.
    x = x0.clone()
    ops.norm_join(x, ops.output_terms([y1], [1.0]), (None, 1.0, eps), T)
    assert (d(x) - (d(x0) + rms(d(y1), eps))).abs().max() < 2e-5 * max(1.0, float(d(x).abs().max()))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("N,W,top", [(6, 96, 2), (64, 768, 8), (1, 32, 1), (33, 50, 4)])
def test_router_with_a_gate_beside_its_experts(dev, dtype, N, W, top):
    from liyab_b200 import ops
    rng = np.random.default_rng(N)
    T = 40
    h = torch.from_numpy(rng.standard_normal((T, W))).to(dtype).to(dev)
    m = torch.from_numpy(rng.standard_normal((N + 1, W)) * 2 * W ** -0.5).to(dtype).to(dev)
    ids, w, gate = torch.empty(T, top, dtype=torch.int32, device=dev), torch.empty(T, top, device=dev), torch.empty(T, device=dev)
    ops.router_choice(ops.router_args(m, top, ids, w, renormalise=True, gate=gate), h)
    z = h.double().cpu() @ m.double().cpu().t()
    wid, ww = choice(z[:, :N], top)
    assert torch.equal(ids.cpu().long(), wid) and (w.double().cpu() - ww).abs().max() < 1e-5
    assert (gate.double().cpu() - torch.sigmoid(z[:, N])).abs().max() < 1e-5
    # Without a gate the last row of a smaller matrix is an expert like the others.
    ops.router_choice(ops.router_args(m[:N].contiguous(), top, ids, w, renormalise=True), h)
    assert torch.equal(ids.cpu().long(), wid)


# ---------------------------------------------------------------- experts without a gate

@pytest.mark.parametrize("act", ["relu2", "silu", "relu"])
@pytest.mark.parametrize("dtype,T,top,E,W,F", [(torch.float32, 9, 2, 5, 60, 24), (torch.float32, 150, 3, 4, 33, 70), (torch.bfloat16, 8, 3, 6, 96, 40), (torch.bfloat16, 90, 2, 7, 136, 72),
                                               (torch.bfloat16, 40, 2, 3, 50, 30), (torch.bfloat16, 300, 1, 5, 64, 8)])
def test_experts_without_a_gate(dev, dtype, T, top, E, W, F, act):
    """Through a plan (32-bit units; a warp a pair; mma.sync tiles), and for a few pairs without one, weights on the input and on the output."""
    from liyab_b200 import ops
    rng = np.random.default_rng(T * F)
    r = lambda *s: torch.from_numpy(rng.standard_normal(s)).to(dtype).to(dev)
    h, up, down = r(T, W), r(E, F, W) * W ** -0.5, r(E, W, F) * F ** -0.5
    ids = torch.from_numpy(np.stack([rng.permutation(E)[:top] for _ in range(T)]).astype(np.int32)).to(dev)
    wts = torch.rand(T, top, device=dev) + 0.5
    f = {"relu2": lambda z: torch.relu(z) ** 2, "silu": torch.nn.functional.silu, "relu": torch.relu}[act]
    d = lambda t: t.double().cpu()
    tol = 2e-5 if dtype == torch.float32 else 4e-2
    for on_input in (False, True):
        want = torch.zeros(T * top, W).double()
        for p in range(T * top):
            e, w = int(ids.flatten()[p]), float(wts.flatten()[p]) if on_input else 1.0
            want[p] = d(down[e]) @ f(w * (d(up[e]) @ d(h[p // top])))
        for plain_units in ([False, True] if dtype == torch.bfloat16 else [False]):
            out = ops.experts_planned(h, up, down, ids, wts if on_input else None, act, plain=True, plain_units=plain_units)
            assert (d(out) - want).abs().max() < tol * max(1.0, float(want.abs().max())), (on_input, plain_units)
        if not on_input and dtype == torch.bfloat16 and T * top <= 64 and W % 8 == 0 and F % 8 == 0:
            out = ops.experts_direct(h, up, down, ids, act, plain=True)
            assert (d(out) - want).abs().max() < tol * max(1.0, float(want.abs().max()))


def test_activations_that_have_no_such_form_are_refused(dev):
    from liyab_b200 import ops
    from liyab_b200.status import LiyabError
    gu = torch.zeros(2, 8, device=dev)
    with pytest.raises(LiyabError):
        ops.gated_act_kind(gu, torch.zeros(2, 4, device=dev), "relu2")


# ---------------------------------------------------------------- the gate on every value

@pytest.mark.parametrize("M,H,E,C", [(5, 3, 14, 24), (70, 4, 32, 64), (64, 12, 64, 256), (200, 2, 70, 10), (1, 1, 1, 1), (33, 5, 8, 40)])
def test_gate_on_every_value_of_the_values_product(dev, M, H, E, C):
    """The product per head with a gate a result on the 32-bit units (both types) and on the tensor cores, with and without the gate, gates that lie in columns of
    a wider buffer."""
    from liyab_b200 import ops
    rng = np.random.default_rng(M * E)
    r = lambda *s: torch.from_numpy(rng.standard_normal(s)).float().to(dev)
    att, uv, wide = r(M, H * C), r(H * E, C) * C ** -0.5, r(M, 7 + H * E)
    gate = wide[:, 7:]
    d = lambda t: t.double().cpu()
    for tb, tc, tensor in ((torch.float32, torch.float32, False), (torch.bfloat16, torch.bfloat16, False), (torch.bfloat16, torch.bfloat16, True)):
        w = uv.to(tb)
        want = torch.einsum("mhc,hec->mhe", d(att).reshape(M, H, C), d(w).reshape(H, E, C)).reshape(M, H * E)
        if tensor and not (C % 8 == 0 and E % 2 == 0):
            continue
        for g in (gate, None):
            out = torch.full((M, H * E), float("nan"), dtype=tc, device=dev)
            ops.head_matmul(att, C, w, E * C, 1, C, out, E, E, C, H, tensor_cores=tensor, gate=g)
            ref = want * torch.sigmoid(d(gate)) if g is not None else want
            assert (d(out) - ref).abs().max() < (1e-5 if tc == torch.float32 else 2e-2) * max(1.0, float(ref.abs().max()))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,F", [(3, 48), (70, 3072), (5, 50), (9, 4), (1, 1), (5000, 8)])
def test_capped_gate_in_pieces_and_value_by_value(dev, dtype, rows, F):
    from liyab_b200 import ops
    rng = np.random.default_rng(rows + F)
    gu = torch.from_numpy(rng.standard_normal((rows, 2 * F)) * 3).float().to(dev)
    out = torch.full((rows, F), float("nan"), dtype=dtype, device=dev)
    ops.gated_act_kind(gu, out, "capped", 1.702, 2.0)
    g, u = gu[:, :F].double().cpu().clamp(max=2.0), gu[:, F:].double().cpu().clamp(-2.0, 2.0)
    want = g * torch.sigmoid(1.702 * g) * (u + 1)
    assert (out.double().cpu() - want).abs().max() < (1e-5 if dtype == torch.float32 else 3e-2)
