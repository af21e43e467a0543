"""Gekitar in the engine against the plain implementation (plain_gekitar.py): every mechanism by itself through the parts' taps, then whole
prompts, token-by-token decoding, portions down to two tokens, mixed batches with pages used again, keys at the windows' edges and at page borders, far
keys, rows shared between layers, the first tokens of a sequence, routed experts, long decoding, and greedy generation through the engine's own entry
point and scheduler."""
from __future__ import annotations

import copy
import os
import subprocess

import numpy as np
import pytest

import plain_gekitar as plain
import trace_tools as tt
from gekitar_models import CONFIGS, attention, dense, f64, latent, layer, model, model_folder, moe, random_weights, to_bf16_values, write_model

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
    base = str(tmp_path_factory.mktemp("gekitar"))
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
    of the sequence's logits; 8 bits of mantissa put it near a percent.  A rounding may send a row to another expert where two scores lie close, and later
    positions see that row: a model with routers may have the share `apart` of its rows beyond `worst`."""
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
TAPS = {"mixer_in": "mixer_norm", "attention": "attention", "heads": "attention", "mixer_out": "mixer.out", "feed_forward_in": "ff_norm",
        "feed_forward_out": "feed_forward.out", "out": "block"}


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_mechanism_by_itself(name, models):
    """The parts' outputs, layer by layer, against the plain functions in float32: the embedded rows, both sublayers' inputs, the attention's heads
    (behind their gate where they have one), both sublayers' outputs before their norm, and the stream after the block.  A whole prompt, then the same prompt cut in two
    and in three."""
    from liyab_b200.engine import StepEntry
    path, config, weights = models[name]
    toks = tokens_of(name, 50, 45)
    want = []
    plain.forward(config, weights, toks, traces=want)
    embedded, want = want[0]["embed"], want[1:]
    L = len(want)
    for cuts in ([len(toks)], [19, len(toks)], [2, 33, len(toks)]):
        engine = make_engine(path, "float32", 128)
        runs = [dict() for _ in want]
        first, seen = [], [0]

        def tap(n, rows):
            if n == "embed":
                first.append(rows)
            elif n != "final_norm":
                if n == "mixer_norm":
                    seen[0] += 1
                runs[(seen[0] - 1) % L].setdefault(n, []).append(rows)
        engine.set_tap(tap)
        engine.cache.open("a")
        lo = 0
        for hi in cuts:
            engine.step([StepEntry("a", toks[lo:hi], [])])
            lo = hi
        assert seen[0] == len(cuts) * L
        assert np.abs(np.concatenate(first, axis=0) - embedded).max() / np.abs(embedded).max() < 2e-6, f"embedded rows (cuts {cuts})"
        for i, ref_run in enumerate(want):
            runs[i]["block"] = runs[i]["feed_forward" if "feed_forward" in runs[i] else "mixer"]      # the stream as the block leaves it
            for plain_name, tap_name in TAPS.items():
                if plain_name not in ref_run or plain_name == ("attention" if "heads" in ref_run else "heads"):        # latent attention: behind its gate
                    continue
                ref = ref_run[plain_name]
                rows = np.concatenate(runs[i][tap_name], axis=0)
                assert rows.shape == ref.shape, (plain_name, rows.shape, ref.shape)
                err = np.abs(rows - ref).max() / max(np.abs(ref).max(), 1e-30)
                assert err < 5e-5, f"{plain_name} of layer {i} (cuts {cuts}): {err:.2e}"


# The share of rows that bfloat16 may send to another expert (A and C choose among many with random routers).
APART = {"A": 0.12, "B": 0.08, "C": 0.12, "D": 0.0}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_cutting_matches_plain(name, dtype, models, oracle):
    path, config, _ = models[name]
    reqs = request_set(name)
    want = oracle[name]
    n_rows = sum(len(t) for t in reqs.values())
    traces = {"whole": tt.whole(reqs), "one_by_one": tt.tail_one_by_one(reqs, 10 ** 6), "tail": tt.tail_one_by_one(reqs, 40),
              "portions": tt.changing_portions(reqs), "odd_portions": tt.changing_portions(reqs, sizes=(2, 31, 2, 17, 1, 3, 33, 16, 2))}
    # D's parts of one value decide by a sign (the norm of a single number is its sign): bfloat16 may flip one, so D is held in float32 only.
    if name == "D" and dtype == "bfloat16":
        pytest.skip("norms over a single value decide by a sign")
    for kind, steps in traces.items():
        engine = make_engine(path, dtype, max_tokens=256)
        got = tt.collect(engine, steps)
        assert len(got) == n_rows
        check(got, want, dtype, apart=APART[name])
    # Mixed batches over a pool for the trace's own peak and four slots for all requests: pages are used again.
    for seed in (3, 4):
        steps = tt.mixed(reqs, max_live=4, seed=seed)
        assert max(len(e) for e, _ in steps) >= 3
        engine = make_engine(path, dtype, max_tokens=tt.peak_tokens(steps, 64))
        got = tt.collect(engine, steps)
        assert len(got) == n_rows
        check(got, want, dtype, apart=APART[name])
        assert len(reqs) > 4 and sum(engine.cache.pages_in_use().values()) == 0


def test_batches_of_unequal_requests_match_each_alone(models):
    """The engine against itself: every request alone and all in mixed batches give the same logits up to rounding."""
    path, _, _ = models["A"]
    reqs = request_set("A")
    alone = tt.collect(make_engine(path, "float32", max_tokens=256), tt.whole(reqs))
    steps = tt.mixed(reqs, max_live=4, seed=11, portion=23)
    together = tt.collect(make_engine(path, "float32", max_tokens=tt.peak_tokens(steps, 64)), steps)
    assert alone.keys() == together.keys()
    scale = max(np.abs(r).max() for r in alone.values())
    assert max(np.abs(alone[k] - together[k]).max() for k in alone) / scale < 2e-5


@pytest.mark.parametrize("page_size", [16, 64])
def test_pages_of_other_sizes(page_size, models, oracle):
    path, _, _ = models["A"]
    engine = make_engine(path, "float32", max_tokens=512, page_size=page_size)
    got = tt.collect(engine, tt.changing_portions(request_set("A"), sizes=(63, 2, 1, 64, 17)))
    check(got, oracle["A"], "float32")


def small(layers, vocab=40, width=32):
    return model(vocab, width, 1e-5, 1.0, layers)


def moved_rows(a, b, by=1e-2):
    return int((np.abs(a - b).max(axis=1) / np.abs(b).max() > by).sum())


def sharp_window_model(base, window, shared):
    """One latent-attention block under a window (`shared`: that reads the rows of a block before it, whose own window is another) whose scores are
    sharpened so that one key takes nearly all the weight: a key that is wrongly seen or wrongly hidden moves the logits by far more than rounding."""
    layers = [layer(latent(2 if window < 40 else 10, 8, 4, 12, 16, 8, 6.0, 100.0, window=window), dense(40, 2.0))]
    if shared:
        layers = [layer(latent(2, 8, 4, 12, 16, 8, 0.2, 100.0, window=shared), dense(24, 2.0)),
                  layer(latent(3, 6, 4, 8, 16, 10, 6.0, 100.0, window=window, kv_from=0), dense(40, 2.0))]
    config = small(layers)
    weights = random_weights(config, 77)
    return write_model(os.path.join(base, f"sharp_{window}_{shared}"), config, weights), config, f64(weights)


@pytest.mark.parametrize("window, shared", [(16, 0), (17, 0), (15, 0), (33, 0), (5, 0), (64, 0), (40, 9), (9, 40), (32, 16)])
def test_window_edges_in_prompts_and_in_decoding(window, shared, tmp_path):
    """Windows that end on, just before and just after page borders, over a block's own rows and over another's whose window is narrower or wider; every
    position of a prompt and of decoding far past the window against the plain model; the plain model with a window one larger or one smaller must
    differ clearly (or the test shows nothing)."""
    path, config, weights = sharp_window_model(str(tmp_path), window, shared)
    toks = np.random.default_rng(5).integers(0, config["vocab"], size=150).astype(int).tolist()
    want = plain.forward(config, weights, toks)
    for delta in (-1, 1):
        other = copy.deepcopy(config)
        other["layers"][-1]["mixer"]["mask"]["size"] += delta
        assert moved_rows(plain.forward(other, weights, toks), want) >= 5, "the weights do not show a window that is one off"
    reqs = {"a": toks}
    for steps in (tt.whole(reqs), tt.tail_one_by_one(reqs, 110), tt.changing_portions(reqs, sizes=(15, 2, 16, 17, 1, 33, 7))):
        for dtype, tol in (("float32", 1e-4), ("bfloat16", None)):
            engine = make_engine(path, dtype, max_tokens=192)
            got = tt.collect(engine, steps)
            if tol is not None:
                tt.check_rows(got, {"a": want}, tol)
            else:
                errs = np.array([np.abs(row - want[pos]).max() for (_, pos), row in got.items()]) / np.abs(want).max()
                assert np.median(errs) < 3e-2 and (errs > 0.2).mean() < 0.05, (np.median(errs), errs.max())
    # The cache unit keeps what the widest reader's window can see, no more: pages behind it came back.
    from liyab_b200.engine import StepEntry
    engine = make_engine(path, "float32", max_tokens=192)
    engine.cache.open("a")
    engine.step([StepEntry("a", toks, [])])
    assert sum(engine.cache.pages_in_use().values()) <= (max(window, shared) + 15) // 16 + 1


def test_what_is_particular_shows(tmp_path):
    """What is particular to the design, each shown by taking it away (or doing it a little differently) on the plain model; the engine agrees with the plain model in
    every cutting and both types."""
    config = small([layer(attention(4, 2, 8, 6, 2.5, 3.0, 6, 50.0, (4.0, 40, 4.0, 0.5)), dense(40, 1.0)), layer(latent(2, 6, 8, 6, 12, 10, 0.9, 50.0), moe(3, 2, 16, 16)),
                    layer(latent(3, 5, 4, 6, 14, 12, 0.8, 20.0, window=30), dense(24, 0.7)),
                    layer(attention(2, 1, 16, 6, 1.0, 8.0, 16, 1000.0, None), None)], width=44)
    weights = random_weights(config, 78)
    weights["l1.mlp.router"] = weights["l1.mlp.router"] * 0.5
    path = write_model(str(tmp_path / "parts"), config, weights)
    weights = f64({k: to_bf16_values(v) for k, v in weights.items()})
    toks = np.random.default_rng(6).integers(0, 40, size=130).astype(int).tolist()
    want = plain.forward(config, weights, toks)

    def swapped(name, other):
        real = getattr(plain, name)
        setattr(plain, name, other)
        try:
            return plain.forward(config, weights, toks)
        finally:
            setattr(plain, name, real)

    def changed(edit):
        other = copy.deepcopy(config)
        edit(other["layers"])
        return plain.forward(other, weights, toks)

    def without(*names):
        return plain.forward(config, {k: v * 0.0 if k in names else v for k, v in weights.items()}, toks)

    real_rotate, real_norm = plain.rotate, plain.zero_centred_norm
    cases = {
        "the cap": swapped("soft_cap", lambda s, cap: s),
        "another cap": swapped("soft_cap", lambda s, cap: 1.3 * cap * np.tanh(s / (1.3 * cap))),
        "the one in the divisor": swapped("softmax_with_one", plain.softmax),
        "the rotation": swapped("rotate", lambda v, pos, rot: v),
        "the stretched frequencies": changed(lambda l: l[0]["mixer"]["rot"].pop("scaling")),
        "where the stretch begins": changed(lambda l: l[0]["mixer"]["rot"]["scaling"].update(fast=1.0)),
        "the factor on cosine and sine": swapped("frequencies", lambda rot, real=plain.frequencies: (real(rot)[0], 1.0)),
        "the bias of q": without("l0.mix.q.b"), "the bias of k": without("l0.mix.k.b"), "the bias of v": without("l0.mix.v.b"), "the bias of o": without("l0.mix.o.b"),
        "the gate's limit": changed(lambda l: l[0]["mlp"].update(limit=1.5)),
        "the norm's offset": swapped("zero_centred_norm", lambda x, w, eps: real_norm(x, w - 1.0, eps)),
        "the shared expert": without("l1.mlp.shared.down"), "its gate": without("l1.mlp.shared.sg"), "the values' gates": without("l1.mix.g"),
        "how many experts": changed(lambda l: l[1]["mlp"]["router"].update(top=1)),
        "the experts' weights": swapped("choose", lambda z, top, real=plain.choose: (real(z, top)[0], np.full(top, 1.0 / top))),
    }
    for what, other in cases.items():
        assert moved_rows(other, want) >= 20, f"{what} does not show"
    reqs = {"a": toks}
    for steps in (tt.whole(reqs), tt.tail_one_by_one(reqs, 100), tt.changing_portions(reqs, sizes=(6, 1, 7, 2, 8, 13, 64))):
        for dtype in ("float32", "bfloat16"):
            check(tt.collect(make_engine(path, dtype, max_tokens=192), steps), {"a": want}, dtype, median=2e-2, worst=0.12, apart=0.1)


def test_the_norm_comes_after_the_rotation(tmp_path):
    """With a factor on cosine and sine that lengthens the rotated part of a head, the order of norm and rotation shows."""
    config = small([layer(attention(2, 1, 12, 8, 3.0, 20.0, 6, 50.0, (300.0, 40, 4.0, 0.5)), dense(40, 1.0))])
    weights = random_weights(config, 12)
    path = write_model(str(tmp_path / "order"), config, weights)
    weights = f64(weights)
    toks = np.random.default_rng(3).integers(0, 40, size=90).astype(int).tolist()
    want = plain.forward(config, weights, toks)
    rotate, rms = plain.rotate, plain.rms
    plain.rotate = lambda v, pos, rot: rotate(rms(v, 1e-5), pos, rot)
    plain.rms = lambda v, eps: v if v.shape[-1] == 12 else rms(v, eps)
    try:
        assert moved_rows(plain.forward(config, weights, toks), want) >= 20, "the order does not show"
    finally:
        plain.rotate, plain.rms = rotate, rms
    for steps in (tt.whole({"a": toks}), tt.tail_one_by_one({"a": toks}, 40), tt.changing_portions({"a": toks})):
        for dtype in ("float32", "bfloat16"):
            check(tt.collect(make_engine(path, dtype, max_tokens=128), steps), {"a": want}, dtype, worst=0.12)


@pytest.mark.parametrize("kind", ["attention", "latent", "shared"])
def test_far_keys(kind, tmp_path):
    """420 tokens under sharpened scores that pick keys hundreds of positions back: whole, decoded (keys cut over blocks), in portions that end on and off page
    borders.  A sequence that lost its first 200 tokens gives clearly different logits (shown on the plain model)."""
    layers = {"attention": [layer(attention(4, 2, 16, 12, 0.6, 9.0, 4, 100.0, (4.0, 100, 8.0, 1.0)), dense(24, 2.0))],
              "latent": [layer(latent(2, 8, 4, 8, 16, 8, 1.5, 100.0), dense(24, 2.0))],
              "shared": [layer(latent(2, 8, 4, 8, 16, 8, 0.3, 100.0, window=20), dense(24, 2.0)),
                         layer(latent(4, 6, 4, 8, 16, 12, 1.5, 100.0, window=300, kv_from=0), dense(24, 2.0))]}[kind]
    config = small(layers, vocab=50)
    weights = random_weights(config, 5)
    path = write_model(str(tmp_path / kind), config, weights)
    weights = f64(weights)
    toks = np.random.default_rng(9).integers(1, 50, size=420).astype(int).tolist()
    want = plain.forward(config, weights, toks)
    lost = {"shared": 110}.get(kind, 200)            # within the window's reach where there is one
    assert moved_rows(plain.forward(config, weights, toks[lost:])[:100], want[lost:lost + 100]) >= 60, "lost tokens do not show"
    reqs = {"a": toks}
    for steps in (tt.whole(reqs), tt.tail_one_by_one(reqs, 30), tt.changing_portions(reqs, sizes=(255, 2, 64, 1, 17))):
        tt.check_rows(tt.collect(make_engine(path, "float32", max_tokens=448), steps), {"a": want}, 2e-4)
    for steps in (tt.whole(reqs), tt.changing_portions(reqs, sizes=(130, 1, 1, 40)), tt.tail_one_by_one(reqs, 60)):
        check(tt.collect(make_engine(path, "bfloat16", max_tokens=448), steps), {"a": want}, "bfloat16", median=2e-2, worst=0.12)


def test_first_tokens_of_a_sequence(tmp_path):
    """Requests of one, two and three tokens and longer ones through ONE slot and a small pool, one after the other: a window's first tokens see only what
    exists, the one in the divisor weighs most where there are few keys, and nothing of the request before is left in the pages."""
    config = small([layer(latent(2, 6, 4, 6, 8, 6, 0.6, 10.0, window=4), None), layer(attention(2, 1, 8, 8, 0.5, 5.0, 8, 10.0), dense(24, 1.0)),
                    layer(latent(2, 4, 4, 4, 8, 6, 0.5), moe(2, 1, 8, 8)), layer(latent(1, 4, 4, 8, 8, 6, 0.7, 10.0, window=7, kv_from=0), None)], vocab=50)
    weights = random_weights(config, 8)
    path = write_model(str(tmp_path / "first"), config, weights)
    weights = f64(weights)
    reqs = {f"r{i}": np.random.default_rng(30 + i).integers(0, 50, size=n).astype(int).tolist() for i, n in enumerate((40, 9, 3, 1, 12, 2))}
    want = {r: plain.forward(config, weights, t) for r, t in reqs.items()}
    for dtype in ("float32", "bfloat16"):
        for steps in (tt.whole(reqs), tt.tail_one_by_one(reqs, 10 ** 6), tt.changing_portions(reqs, sizes=(1, 1, 2, 1, 3, 2, 17))):
            got = tt.collect(make_engine(path, dtype, max_tokens=64, max_requests=1), steps)
            check(got, want, dtype, median=2e-2, worst=8e-2, apart=0.08)


def test_a_router_that_decides_clearly(tmp_path):
    """Routers that send tokens by a few strong coordinates of the stream: both types choose alike on every row, so every row is held."""
    config = small([layer(latent(2, 4, 4, 4, 8, 6, 0.5), moe(6, 2, 24, 16)), layer(attention(1, 1, 8, 8, 0.5, 5.0, 8, 10.0), moe(6, 6, 8))], vocab=30, width=48)
    weights = random_weights(config, 7)
    weights["embed"][:, :6] = np.random.default_rng(8).choice([-4.0, 4.0], size=(30, 6)) * np.array([1.0, 1.2, 1.4, 1.6, 1.8, 2.0])
    weights["l0.mlp.router"] = np.zeros((6, 48))
    weights["l0.mlp.router"][:, :6] = np.eye(6) * 1.5
    weights["l0.norm1b"] = weights["l0.norm1b"] * 0.0 - 0.8          # the mixer moves the stream little
    path = write_model(str(tmp_path / "clear"), config, weights)
    weights = f64({k: to_bf16_values(v) for k, v in weights.items()})
    toks = np.random.default_rng(2).integers(0, 30, size=100).astype(int).tolist()
    traces = []
    want = plain.forward(config, weights, toks, traces)
    z = np.sort(traces[1]["router"], axis=1)
    assert (z[:, -2] - z[:, -3]).min() > 0.05 and len(np.unique(traces[1]["chosen"])) >= 5
    for steps in (tt.whole({"a": toks}), tt.changing_portions({"a": toks}, sizes=(20, 1, 2, 9)), tt.tail_one_by_one({"a": toks}, 60)):
        for dtype in ("float32", "bfloat16"):
            check(tt.collect(make_engine(path, dtype, max_tokens=128), steps), {"a": want}, dtype)


def test_long_decoding_reuses_pages(models):
    """Decoding one token at a time far past every window: pages are freed behind the windows and handed out again."""
    path, config, weights = models["A"]
    toks = tokens_of("A", 99, 400)
    want = plain.forward(config, weights, toks)
    engine = make_engine(path, "float32", max_tokens=448)       # full caches stay; the windows' pages go round
    got = tt.collect(engine, tt.tail_one_by_one({"a": toks}, 395))
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
    check(got, oracle["A"], dtype, apart=APART["A"])


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_engine(graphs, models):
    """Prompts of unequal length served together by the scheduler, greedy, against the plain model's own greedy continuation (compared
    while the plain model's best two logits are clearly apart)."""
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
    """The command line generates greedily what the plain model would, and the engine's sampler with a seed gives the same tokens twice
    and other tokens with another seed."""
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
