"""Mokisun in the engine against the plain implementation (plain_mokisun.py): every mechanism by itself through the parts' taps, then whole
prompts, token-by-token decoding, portions down to two tokens, mixed batches with pages and state slots used again, keys at the windows' edges and at
page borders, slopes and divisors, memories that reach far back and that forget at once, the first tokens of a sequence, corrected and grouped routing,
long decoding, and greedy generation through the engine's own entry point and scheduler."""
from __future__ import annotations

import copy
import os
import subprocess

import numpy as np
import pytest

import plain_mokisun as plain
import trace_tools as tt
from mokisun_models import CONFIGS, attention, delta, f64, gla, keyed, layer, model, model_folder, moe, parallel, random_weights, write_model

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# float32: largest |engine - plain| on a logit as a fraction of the largest |logit| of the sequence.
REL_TOL = 1e-4
LENGTHS = {"A": [150, 70, 33, 21, 7, 2, 1, 45], "B": [140, 72, 64, 1, 2, 97, 40], "C": [120, 47, 2, 64, 1, 33], "D": [100, 33, 32, 31, 2, 65]}


def tokens_of(name, i, n):
    config, seed = CONFIGS[name]
    return np.random.default_rng(1000 * seed + i).integers(0, config["vocab"], size=n).astype(int).tolist()


def request_set(name):
    return {f"r{i}": tokens_of(name, i, n) for i, n in enumerate(LENGTHS[name])}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    base = str(tmp_path_factory.mktemp("mokisun"))
    out = {}
    for name in CONFIGS:
        path, config, weights = model_folder(base, name)
        out[name] = (path, config, f64(weights))
    return out


@pytest.fixture(scope="module")
def oracle(models):
    return {name: {r: plain.forward(config, weights, toks) for r, toks in request_set(name).items()}
            for name, (_, config, weights) in models.items()}


def make_engine(path, dtype, max_tokens, **options):
    from liyab_b200.engine import Replayer
    options.setdefault("max_requests", 4)
    return Replayer(path, dtype, max_tokens, **options)


def check(got, want, dtype, rel_tol=REL_TOL, median=1.5e-2, worst=6e-2, apart=0.0):
    """float32: every logit within rel_tol of the plain model's.  bfloat16: per row, the root mean square of the difference (its mean taken off) over that
    of the sequence's logits; 8 bits of mantissa put it near a percent.  A rounding may send a row to another expert where two choice scores lie close,
    and memories carry that on: a model with routers may have the share `apart` of its rows beyond `worst`."""
    if dtype != "bfloat16":
        return tt.check_rows(got, want, rel_tol)
    errs = []
    for (r, pos), row in got.items():
        d = row.astype(np.float64) - want[r][pos]
        spread = want[r] - want[r].mean(axis=-1, keepdims=True)
        errs.append(np.sqrt(((d - d.mean()) ** 2).mean()) / np.sqrt((spread ** 2).mean()))
    errs = np.asarray(errs)
    assert np.isfinite(errs).all() and np.median(errs) <= median, f"median relative error {np.median(errs):.3e}"
    assert (errs > worst).mean() <= apart, f"{(errs > worst).sum()} of {len(errs)} rows are off by more than {worst}, the worst by {errs.max():.3f}"
    return {"mean": float(errs.mean()), "worst": float(errs.max())}


# What the plain model calls a part's output -> the name of the engine's tap.
TAPS = {"attention": "attention", "memory": "memory", "heads": "memory.heads", "left": "branch.left", "right": "branch.right"}


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_mechanism_by_itself(name, models):
    """The parts' outputs, layer by layer, against the plain functions in float32: the attention's heads, what the memories give before their norm and
    gate and after, both sides of a pair, and all streams after the mixer and after the block.  A whole prompt, then the same prompt cut in two, in
    three and in portions short enough for the row-by-row form."""
    from liyab_b200.engine import StepEntry
    path, config, weights = models[name]
    toks = tokens_of(name, 50, 45)
    want = []
    plain.forward(config, weights, toks, traces=want)
    for cuts in ([len(toks)], [19, len(toks)], [2, 33, len(toks)], [13, 15, 16, 30, 31, len(toks)]):
        engine = make_engine(path, "float32", 128)
        runs = [dict() for _ in want]
        at = [-1]

        def tap(n, rows):
            if n == "mixer_norm":                  # a block begins
                at[0] += 1
            if n not in ("embed", "final_norm"):
                runs[at[0] % len(want)].setdefault(n, []).append(rows)
        engine.set_tap(tap)
        engine.cache.open("a")
        lo = 0
        for hi in cuts:
            engine.step([StepEntry("a", toks[lo:hi], [])])
            lo = hi
        assert at[0] + 1 == len(cuts) * len(want)
        for i, ref in enumerate(want):
            expected = {TAPS[k]: v for k, v in ref.items() if k in TAPS}
            expected["mixer"] = ref["mixer"].reshape(len(toks), -1)
            expected["feed_forward" if config["layers"][i]["mlp"] else "mixer"] = ref["out"].reshape(len(toks), -1)
            for tap_name, value in expected.items():
                rows = np.concatenate(runs[i][tap_name], axis=0)
                assert rows.shape == value.shape, (tap_name, rows.shape, value.shape)
                err = np.abs(rows - value).max() / max(np.abs(value).max(), 1e-30)
                assert err < 5e-5, f"{tap_name} of layer {i} (cuts {cuts}): {err:.2e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_cutting_matches_plain(name, dtype, models, oracle):
    path, config, _ = models[name]
    reqs = request_set(name)
    want = oracle[name]
    n_rows = sum(len(t) for t in reqs.values())
    traces = {"whole": tt.whole(reqs), "one_by_one": tt.tail_one_by_one(reqs, 10 ** 6), "tail": tt.tail_one_by_one(reqs, 40),
              "portions": tt.changing_portions(reqs), "odd_portions": tt.changing_portions(reqs, sizes=(2, 31, 2, 17, 1, 3, 33, 16, 2))}
    # D's norms over a single value decide by a sign: bfloat16 may flip one, so D is held in float32 only.
    if name == "D" and dtype == "bfloat16":
        pytest.skip("norms over a single value decide by a sign")
    for kind, steps in traces.items():
        engine = make_engine(path, dtype, max_tokens=256)
        got = tt.collect(engine, steps)
        assert len(got) == n_rows
        check(got, want, dtype, median=2e-2, apart=0.1)
    # Mixed batches over a pool for the trace's own peak and four state slots for all requests: pages and slots are used again.
    for seed in (3, 4):
        steps = tt.mixed(reqs, max_live=4, seed=seed)
        assert max(len(e) for e, _ in steps) >= 3
        engine = make_engine(path, dtype, max_tokens=tt.peak_tokens(steps, 64))
        got = tt.collect(engine, steps)
        assert len(got) == n_rows
        check(got, want, dtype, median=2e-2, apart=0.1)
        assert len(reqs) > 4 and engine.cache.state_slots_free() == 4


def test_batches_of_unequal_requests_match_each_alone(models):
    """The engine against itself: every request alone and all in mixed batches give the same logits up to rounding."""
    path, _, _ = models["A"]
    reqs = request_set("A")
    alone = tt.collect(make_engine(path, "float32", max_tokens=256), tt.whole(reqs))
    steps = tt.mixed(reqs, max_live=4, seed=11, portion=23)
    together = tt.collect(make_engine(path, "float32", max_tokens=tt.peak_tokens(steps, 64)), steps)
    assert alone.keys() == together.keys()
    scale = max(np.abs(r).max() for r in alone.values())
    assert max(np.abs(alone[k] - together[k]).max() for k in alone) / scale < 3e-5


@pytest.mark.parametrize("page_size", [16, 64])
def test_pages_of_other_sizes(page_size, models, oracle):
    path, _, _ = models["A"]
    engine = make_engine(path, "float32", max_tokens=512, page_size=page_size)
    got = tt.collect(engine, tt.changing_portions(request_set("A"), sizes=(63, 2, 1, 64, 17)))
    check(got, oracle["A"], "float32")


def small(layers, vocab=40, width=32, streams=2):
    return model(vocab, width, streams, 1e-5, layers)


def moved_rows(a, b, by=1e-2):
    return int((np.abs(a - b).max(axis=1) / np.abs(b).max() > by).sum())


def sharp_window_model(base, window, kind, kv_heads=1):
    """One block whose scores are sharpened so that one key takes nearly all the weight: a key that is wrongly seen or wrongly hidden moves the logits by
    far more than rounding.  In a pair the delta side is silenced and the slopes of many heads are small, so that far keys still count."""
    if kind == "rotary":
        config = small([layer(attention(2, kv_heads, 8, 12, 5.0, window, 4, 100.0), None)])
    else:
        config = small([layer(parallel(keyed(8, kv_heads, 8, 5.0, window), delta(1, 1, 4, 4, 2), 1.0, 0.0), None)], vocab=160)
    weights = random_weights(config, 77)
    if kind == "rotary":
        weights["l0.mix.sink"] = np.zeros(2)
    return write_model(os.path.join(base, f"sharp_{kind}_{window}_{kv_heads}"), config, weights), config, f64(weights)


@pytest.mark.parametrize("kind", ["rotary", "keyed"])
@pytest.mark.parametrize("window", [16, 17, 15, 33, 5, 64])
def test_window_edges_in_prompts_and_in_decoding(window, kind, tmp_path):
    """Windows that end on, just before and just after page borders; every position of a prompt and of decoding far past the window against the plain
    model; the plain model with a window one larger or one smaller must differ clearly (or the test shows nothing)."""
    path, config, weights = sharp_window_model(str(tmp_path), window, kind, kv_heads=2 if window == 33 else 1)
    rng = np.random.default_rng(5)       # in a pair every token comes once: a nearer copy of a key would outweigh it by the slopes
    toks = (rng.integers(0, config["vocab"], size=150) if kind == "rotary" else rng.permutation(160)[:150]).astype(int).tolist()
    want = plain.forward(config, weights, toks)
    for d in (-1, 1):
        other = copy.deepcopy(config)
        m = other["layers"][0]["mixer"]
        (m if kind == "rotary" else m["left"])["mask"]["size"] += d
        assert moved_rows(plain.forward(other, weights, toks), want) >= 5, "the weights do not show a window that is one off"
    reqs = {"a": toks}
    for steps in (tt.whole(reqs), tt.tail_one_by_one(reqs, 110), tt.changing_portions(reqs, sizes=(15, 2, 16, 17, 1, 33, 7))):
        for dtype, tol in (("float32", 1e-4), ("bfloat16", None)):
            got = tt.collect(make_engine(path, dtype, max_tokens=192), steps)
            if tol is not None:
                tt.check_rows(got, {"a": want}, tol)
            else:
                errs = np.array([np.abs(row - want[pos]).max() for (_, pos), row in got.items()]) / np.abs(want).max()
                assert np.median(errs) < 2e-2 and (errs > 0.15).mean() < 0.05, (np.median(errs), errs.max())
    # The cache unit keeps what the window can see, no more: pages behind it came back.
    from liyab_b200.engine import StepEntry
    engine = make_engine(path, "float32", max_tokens=192)
    engine.cache.open("a")
    engine.step([StepEntry("a", toks, [])])
    assert sum(engine.cache.pages_in_use().values()) <= (window + 15) // 16 + 1


def test_what_is_particular_shows(tmp_path):
    """Each particular piece shown by taking it away on the plain model; the engine agrees with the plain model in every cutting and both types: the
    sink and that it is not scaled, the rotation and its pairing, the slopes, the one in the divisor, the two sides' factors, the convolution, the unit
    vectors, the delta rule's rate, the decay by channel, the order of decay and write, the mixing of the streams (from, to)."""
    config = small([layer(attention(3, 1, 8, 6, 1.5, 40, 6, 50.0), None), layer(parallel(keyed(4, 2, 8, 1.0, 30), delta(4, 2, 6, 10, 3), 0.8, 1.4), None),
                    layer(gla(2, 8, 8, 2.0), None)], width=44, streams=3)
    weights = random_weights(config, 78)
    weights["l0.mix.sink"] = np.array([2.0, -1.0, 3.0])
    weights["l0.hc1.out"] = np.array([1.5, -0.5, 0.75])
    weights["l1.hc1.mix"] = np.array([[0.625, 0.75, 0.0], [-0.5, 0.75, 0.5], [0.0, 0.125, 0.5]])
    path = write_model(str(tmp_path / "parts"), config, weights)
    weights = f64(weights)
    toks = np.random.default_rng(6).integers(0, 40, size=130).astype(int).tolist()
    want = plain.forward(config, weights, toks)

    def swapped(name, other):
        real = getattr(plain, name)
        setattr(plain, name, other)
        try:
            return plain.forward(config, weights, toks)
        finally:
            setattr(plain, name, real)

    def reset(**changes):
        changed = dict(weights)
        changed.update({k.replace("__", "."): v for k, v in changes.items()})
        return plain.forward(config, changed, toks)

    softmax, rotate, conv, memory, linear = plain.weights_with_sink, plain.rotate_pairs, plain.causal_conv, plain.delta_memory, plain.gated_linear
    shown = {
        "sinks": swapped("weights_with_sink", lambda s, sink: softmax(s, -1e30)),
        "a scaled sink": swapped("weights_with_sink", lambda s, sink: softmax(s, sink * 1.5)),
        "the one in the divisor": swapped("weights_with_sink", lambda s, sink: softmax(s, sink if sink != 0 else -1e30)),
        "the rotation": swapped("rotate_pairs", lambda v, rot: v),
        "its pairing": swapped("rotate_pairs", lambda v, rot: rotate(v[..., [0, 3, 1, 4, 2, 5, 6, 7]], rot)[..., [0, 2, 4, 1, 3, 5, 6, 7]]),
        "the slopes": swapped("head_slopes", lambda H: np.zeros(H)),
        "the convolution": swapped("causal_conv", lambda x, taps: conv(x, taps[:, ::-1])),
        "the unit vectors": swapped("unit", lambda v: v),
        "the rate": swapped("delta_memory", lambda q, k, v, g, b: memory(q, k, v, g, np.ones_like(b))),
        "the rule": swapped("delta_memory", lambda q, k, v, g, b: linear(np.repeat(q, 2, 1), np.repeat(k, 2, 1), b[..., None] * v, g)),
        "the decay by channel": swapped("gated_linear", lambda q, k, v, a: linear(q, k, v, np.broadcast_to(a.mean(-1, keepdims=True), a.shape))),
        "the mixing's direction": reset(l1__hc1__mix=weights["l1.hc1.mix"].T),
        "the layer scale": reset(l1__ls1=np.ones(44)),
        "the norm's alpha": reset(l2__norm1__alpha=weights["l2.norm1.alpha"] * 1.2),
    }
    for what, other in shown.items():
        assert moved_rows(other, want) >= 50, f"{what}: does not show"
    reqs = {"a": toks}
    for steps in (tt.whole(reqs), tt.tail_one_by_one(reqs, 100), tt.changing_portions(reqs, sizes=(6, 1, 7, 2, 8, 13, 64))):
        for dtype in ("float32", "bfloat16"):       # scores this sharp double what a rounding of a query or key costs
            check(tt.collect(make_engine(path, dtype, max_tokens=192), steps), {"a": want}, dtype, median=2e-2, worst=0.12)


def slow_memories(weights, config):
    for i, l in enumerate(config["layers"]):
        if l["type"] == "gla":
            weights[f"l{i}.mix.a2.b"] = np.full_like(weights[f"l{i}.mix.a2.b"], 7.0)
        elif l["type"] == "parallel":
            weights[f"l{i}.mix.right.A_log"] = np.full_like(weights[f"l{i}.mix.right.A_log"], -5.0)
            weights[f"l{i}.mix.right.dt_bias"] = np.full_like(weights[f"l{i}.mix.right.dt_bias"], -2.0)
            weights[f"l{i}.mix.right.b"] = weights[f"l{i}.mix.right.b"] * 0.1 - 0.35 / 32          # small rates: old entries are not overwritten
    return weights


def test_far_keys_and_memories_that_reach_far_back(tmp_path):
    """420 tokens: a wide window whose sharpened scores pick keys hundreds of positions back, and memories that forget slowly.  Whole (a block per piece of the
    prompt), decoded (row by row), in portions that end on and off page borders.  A sequence that lost its first 200 tokens gives clearly different
    logits in each layer alone (shown on the plain model)."""
    layers = [layer(gla(4, 8, 12, 10.0), None), layer(attention(2, 1, 8, 8, 2.5, 1000, 4, 100.0), None),
              layer(parallel(keyed(2, 1, 8, 0.3, 6), delta(2, 1, 24, 12, 3), 0.3, 1.5), None)]
    toks = np.random.default_rng(9).integers(1, 50, size=420).astype(int).tolist()
    for i, one in enumerate(layers):
        config = small([one], vocab=50)
        weights = f64(slow_memories(random_weights(config, 5 + i), config))
        lost = moved_rows(plain.forward(config, weights, toks[200:]), plain.forward(config, weights, toks)[200:])
        assert lost >= (100 if i == 1 else 60), f"layer {i} does not show lost tokens ({lost})"
    config = small(layers, vocab=50)
    weights = slow_memories(random_weights(config, 5), config)
    path = write_model(str(tmp_path / "far"), config, weights)
    from mokisun_models import to_bf16_values
    weights = f64({k: to_bf16_values(v) for k, v in weights.items()})
    want = plain.forward(config, weights, toks)
    reqs = {"a": toks}
    for steps in (tt.whole(reqs), tt.tail_one_by_one(reqs, 30), tt.changing_portions(reqs, sizes=(255, 2, 64, 1, 17))):
        tt.check_rows(tt.collect(make_engine(path, "float32", max_tokens=448), steps), {"a": want}, 2e-4)
    for steps in (tt.changing_portions(reqs, sizes=(130, 1, 1, 40)), tt.tail_one_by_one(reqs, 60)):
        check(tt.collect(make_engine(path, "bfloat16", max_tokens=448), steps), {"a": want}, "bfloat16", median=2e-2, worst=8e-2)


def test_memories_that_forget_at_once(tmp_path):
    """Decays so strong that a piece's running sum of logarithms reaches hundreds: nothing overflows, nothing turns into a number that is none, and what is kept
    (channels that decay slowly beside channels that are wiped by every token) is right in pieces and row by row."""
    config = small([layer(gla(2, 16, 8, 0.05), None), layer(parallel(keyed(2, 1, 8, 0.3, 6), delta(2, 2, 16, 12, 3), 0.3, 1.5), None)])
    weights = random_weights(config, 15)
    rng = np.random.default_rng(16)
    weights["l0.mix.a2.b"] = rng.choice([-3.0, 0.5, 6.0, 9.0], size=weights["l0.mix.a2.b"].shape)
    weights["l1.mix.right.A_log"] = np.array([3.0, -3.0])
    weights["l1.mix.right.dt_bias"] = rng.choice([2.0, -1.0, -8.0], size=weights["l1.mix.right.dt_bias"].shape)
    path = write_model(str(tmp_path / "fast"), config, weights)
    weights = f64(weights)
    toks = rng.integers(0, 40, size=140).astype(int).tolist()
    reqs = {"a": toks}
    want = plain.forward(config, weights, toks)
    for steps in (tt.whole(reqs), tt.tail_one_by_one(reqs, 70), tt.changing_portions(reqs, sizes=(33, 2, 64, 1, 17))):
        tt.check_rows(tt.collect(make_engine(path, "float32", max_tokens=192), steps), {"a": want}, 2e-4)
        check(tt.collect(make_engine(path, "bfloat16", max_tokens=192), steps), {"a": want}, "bfloat16", median=2e-2, worst=8e-2)


def test_first_tokens_of_a_sequence(tmp_path):
    """Requests of one, two and three tokens and longer ones through ONE state slot and a small pool, one after the other: a memory starts at zero, a
    convolution's inputs before the start are zeros, the one in the divisor weighs most where there are few keys, and nothing of the request before is left
    in the slot or the pages."""
    config = small([layer(gla(2, 8, 6, 20.0), None), layer(parallel(keyed(2, 1, 8, 0.5, 4), delta(2, 2, 8, 6, 4), 1.0, 1.0), None),
                    layer(attention(1, 1, 8, 8, 0.5, 7, 2, 10.0), None), layer(parallel(keyed(1, 1, 8, 0.5, 9), delta(3, 1, 5, 6, 7), 1.0, 1.0), None)], vocab=50)
    weights = random_weights(config, 8)
    path = write_model(str(tmp_path / "first"), config, weights)
    weights = f64(weights)
    reqs = {f"r{i}": np.random.default_rng(30 + i).integers(0, 50, size=n).astype(int).tolist() for i, n in enumerate((40, 9, 3, 1, 12, 2))}
    want = {r: plain.forward(config, weights, t) for r, t in reqs.items()}
    for dtype in ("float32", "bfloat16"):
        for steps in (tt.whole(reqs), tt.tail_one_by_one(reqs, 10 ** 6), tt.changing_portions(reqs, sizes=(1, 1, 2, 1, 3, 2, 17))):
            got = tt.collect(make_engine(path, dtype, max_tokens=64, max_requests=1), steps)
            check(got, want, dtype, median=2e-2, worst=8e-2)


def test_corrected_choices_groups_and_identities(tmp_path):
    """Routers whose choices are far apart (the gaps are checked on the plain model), so that both types must choose alike: the correction in the choice and
    not in the weight, the groups, the identities and the factor each show on the plain model by being taken away."""
    config = small([layer(gla(2, 8, 8, 10.0), moe(7, 3, 24, identity=2, groups=3, keep=2, scale=2.5)), layer(attention(2, 2, 8, 8, 0.4, 12, 8), moe(4, 2, 16, identity=2)),
                    layer(gla(1, 8, 8, 10.0), moe(3, 1, 8, identity=3, groups=2, keep=1, scale=3.0))], vocab=40, width=48)
    weights = random_weights(config, 101)
    rng = np.random.default_rng(3)
    for i in range(3):            # scores far apart: the routers read a few strong directions of their own
        weights[f"l{i}.mlp.router"] = weights[f"l{i}.mlp.router"] * 2.0
        weights[f"l{i}.mlp.correction"] = rng.uniform(-1.6, -1.0, size=weights[f"l{i}.mlp.correction"].shape)
    path = write_model(str(tmp_path / "routers"), config, weights)
    from mokisun_models import to_bf16_values
    weights = f64({k: to_bf16_values(v) for k, v in weights.items()})
    toks = np.random.default_rng(27).integers(0, 40, size=90).astype(int).tolist()
    traces = []
    want = plain.forward(config, weights, toks, traces)
    counts = np.bincount(np.concatenate([t["chosen"].ravel() for t in traces[:1]]), minlength=9)
    assert (counts[:7] > 0).sum() >= 3 and counts[7:].sum() > 0, counts

    def changed(i, **router):
        other = copy.deepcopy(config)
        other["layers"][i]["mlp"]["router"].update(router)
        return plain.forward(other, weights, toks)

    assert moved_rows(changed(0, groups=dict(count=3, keep=3)), want) >= 5, "the groups do not show"
    assert moved_rows(changed(0, scale=2.4), want) >= 20, "the factor does not show"
    flat = dict(weights)
    flat["l0.mlp.correction"] = np.zeros(9)
    assert moved_rows(plain.forward(config, flat, toks), want) >= 20, "the correction does not show"
    real = plain.experts_ff

    def corrected_weights(h, W, p, mlp, trace=None):
        r = mlp["router"]
        W2 = dict(W)
        y = real(h, W2, p, mlp, trace)
        return y + 0.1 * sum(W[p + "correction"][:1]) * h * (r["identity"] > 0)
    plain.experts_ff = corrected_weights
    try:
        assert moved_rows(plain.forward(config, weights, toks), want) >= 20, "what the identities add does not show"
    finally:
        plain.experts_ff = real
    for steps in (tt.whole({"a": toks}), tt.changing_portions({"a": toks}, sizes=(20, 1, 2, 9)), tt.tail_one_by_one({"a": toks}, 60)):
        check(tt.collect(make_engine(path, "float32", max_tokens=128), steps), {"a": want}, "float32")
        check(tt.collect(make_engine(path, "bfloat16", max_tokens=128), steps), {"a": want}, "bfloat16", median=2e-2, apart=0.12)


def test_a_router_that_decides_clearly(tmp_path):
    """One block whose router sends tokens by one strong coordinate of the stream: both types choose alike on every row, so every row is held."""
    config = small([layer(gla(2, 8, 8, 10.0), moe(4, 2, 24, identity=2, groups=3, keep=2, scale=2.0))], vocab=30, width=48)
    weights = random_weights(config, 7)
    pattern = np.random.default_rng(8).choice([-3.0, 3.0], size=(30, 6))
    weights["embed"][:, :6] = pattern
    weights["l0.mlp.router"] = np.zeros((6, 48))
    weights["l0.mlp.router"][:, :6] = np.eye(6) * np.array([1.0, 1.3, 1.6, 1.9, 2.2, 2.5])[:, None]
    weights["l0.mlp.correction"] = np.array([-0.5, -0.45, -0.4, -0.3, -0.2, -0.6])
    weights["l0.ls1"] = weights["l0.ls1"] * 0.2
    path = write_model(str(tmp_path / "clear"), config, weights)
    from mokisun_models import to_bf16_values
    weights = f64({k: to_bf16_values(v) for k, v in weights.items()})
    toks = np.random.default_rng(2).integers(0, 30, size=100).astype(int).tolist()
    want = plain.forward(config, weights, toks)
    for steps in (tt.whole({"a": toks}), tt.changing_portions({"a": toks}, sizes=(20, 1, 2, 9)), tt.tail_one_by_one({"a": toks}, 60)):
        for dtype in ("float32", "bfloat16"):
            check(tt.collect(make_engine(path, dtype, max_tokens=128), steps), {"a": want}, dtype, apart=0.03)


def test_long_decoding_reuses_pages(models):
    """Decoding one token at a time far past every window: pages are freed behind the windows and handed out again, and the memories run through 400 single
    steps over a pool that could not hold the sequence."""
    path, config, weights = models["A"]
    toks = tokens_of("A", 99, 400)
    want = plain.forward(config, weights, toks)
    got = tt.collect(make_engine(path, "float32", max_tokens=128), tt.tail_one_by_one({"a": toks}, 395))
    assert len(got) == 400
    tt.check_rows(got, {"a": want}, 2e-4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(dtype, models, oracle, tmp_path):
    path, config, _ = models["A"]
    reqs = request_set("A")
    steps = tt.mixed(reqs, max_live=4, seed=8)
    out_dir = str(tmp_path / "out")
    proc = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", out_dir,
                           "--max-tokens", str(tt.peak_tokens(steps))], input=tt.to_jsonl(steps), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    held, got = {}, {}
    for i, (entries, end) in enumerate(steps):
        data = np.fromfile(os.path.join(out_dir, f"{i}.f32"), dtype="<f4").reshape(-1, config["vocab"])
        row = 0
        for r, toks, want in entries:
            base = held.get(r, 0)
            for w in want:
                got[(r, base + w)] = data[row]
                row += 1
            held[r] = base + len(toks)
        assert row == data.shape[0]
    check(got, oracle["A"], dtype, median=2e-2, apart=0.1)


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_engine(graphs, models):
    """Prompts of unequal length served together by the scheduler, greedy, against the plain model's own greedy continuation (compared while the plain
    model's best two logits are clearly apart)."""
    from liyab_b200.engine import Engine
    from liyab_b200.sampling import SamplingParams
    path, config, weights = models["A"]
    prompts = [tokens_of("A", 70 + i, n) for i, n in enumerate((37, 5, 1, 64, 18, 90))]
    engine = Engine(model=path, dtype="float32", context_length=256, max_requests=4, max_batched_tokens=48, cuda_graphs=graphs)
    results = engine.generate_batch(prompts, SamplingParams(max_tokens=24, temperature=0.0))
    engine.close()
    for prompt, res in zip(prompts, results):
        assert res.error is None and len(res.tokens) == 24
        seq = list(prompt)
        for tok in res.tokens:
            row = plain.forward(config, weights, seq)[-1]
            best = np.sort(row)[-2:]
            if best[1] - best[0] < 1e-3 * np.abs(row).max():
                break
            assert tok == int(np.argmax(row))
            seq.append(tok)


def test_command_line_and_sampling(models):
    """The command line generates greedily what the plain model would, and the engine's sampler with a seed gives the same tokens twice and other tokens with
    another seed."""
    import json
    from liyab_b200.engine import Engine
    from liyab_b200.sampling import SamplingParams
    path, config, weights = models["B"]
    prompt = tokens_of("B", 90, 9)
    cmd = [os.path.join(ROOT, "bin", "liyab-cli"), "-m", path, "-p", ",".join(map(str, prompt)), "-n", "8", "--temp", "0", "--dtype", "float32",
           "--ctx", "128", "--json"]
    proc = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    lines = [json.loads(l) for l in proc.stdout.splitlines() if l.startswith("{")]
    seq = list(prompt)
    for tok in lines[1]["tokens"]:
        row = plain.forward(config, weights, seq)[-1]
        best = np.sort(row)[-2:]
        if best[1] - best[0] < 1e-3 * np.abs(row).max():
            break
        assert tok == int(np.argmax(row))
        seq.append(tok)
    draws = []
    for seed in (5, 5, 6):
        engine = Engine(model=path, dtype="bfloat16", context_length=128, max_requests=4)
        draws.append(engine.generate_tokens(prompt, SamplingParams(max_tokens=12, temperature=0.9, top_k=20, top_p=0.95, seed=seed)).tokens)
        engine.close()
    assert draws[0] == draws[1] and draws[0] != draws[2] and all(0 <= t < config["vocab"] for t in draws[2])
