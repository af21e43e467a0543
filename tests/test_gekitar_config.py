"""Gekitar's configuration, model description, checkpoint map and cache needs, without a GPU."""
from __future__ import annotations

import copy

import numpy as np
import pytest

import plain_gekitar as plain
from gekitar_models import CONFIG_A, CONFIG_B, CONFIG_C, CONFIG_D, random_weights, rotation, write_model
from liyab_b200.config import describe_config, slot, supported_architectures
from liyab_b200.status import LiyabError


def test_registered_and_found_by_its_own_key():
    assert "gekitar" in supported_architectures()
    assert describe_config(CONFIG_A)["architecture"] == "gekitar"


@pytest.mark.parametrize("config", [CONFIG_A, CONFIG_B, CONFIG_C, CONFIG_D])
def test_every_size_and_constant_comes_from_the_file(config):
    d = describe_config(config)["spec"]
    W, eps = config["width"], config["norm"]["eps"]
    norm = {"kind": "rms_norm", "size": W, "groups": 1, "eps": eps, "gain_offset": 1.0}
    assert d["embedding"] == {"vocab_size": config["vocab"], "size": W, "scale": config["embedding"]["scale"]}
    assert not d["head"]["tied"] and d["head"]["logit_scale"] == 1.0 and d["position"]["kind"] == "none" and d["final_norm"] == norm
    assert [(e["layer"], e["cache"]) for e in d["run_order"]] == [(i, l["mixer"].get("kv_from", i)) for i, l in enumerate(config["layers"])]
    for layer, raw in zip(d["layers"], config["layers"]):
        assert layer["arrangement"] == "sandwich_norm"
        names = [s["name"] for s in layer["slots"]]
        assert names == ["mixer_norm", "mixer", "mixer_out_norm"] + (["ff_norm", "feed_forward", "ff_out_norm"] if raw["mlp"] else [])
        assert all(slot(layer, n) == norm for n in names if n.endswith("norm"))
        m, r = slot(layer, "mixer"), raw["mixer"]
        if raw["type"] == "attention":
            assert m["kind"] == "gated_attention" and m["bias"] and m["out_bias"] and m["gate"] == "none" and m["unit_sink"] and m["window"] == 0
            assert m["qk_norm"] and not m["qk_gain"] and m["qk_norm_at"] == "rotated" and m["rot_layout"] == "interleaved" and m["eps"] == eps
            assert (m["n_head"], m["n_kv_head"], m["dim"], m["vdim"], m["scale"], m["soft_cap"]) == (r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["scale"], r["softcap"])
            assert (m["rot_dims"], m["rot_base"], m.get("rot_scaling")) == (r["rot"]["dims"], r["rot"]["base"], r["rot"].get("scaling"))
        else:
            assert m["kind"] == "latent_attention" and m["rot_layout"] == "interleaved" and m["own_latent"] == ("kv_from" not in r)
            assert m["value_gate"] == (raw["type"] == "latent_attention") and m["window"] == (r["mask"]["size"] if "mask" in r else 0)
            assert (m["n_head"], m["dim"], m["rot_dim"], m["rot_dims"], m["vdim"], m["kv_rank"], m["q_rank"], m["scale"], m["rot_base"], m["eps"]) == (
                r["heads"], r["dim"], r["rot_dim"], r["rot"]["dims"], r["vdim"], r["kv_rank"], r["q_rank"], r["scale"], r["rot"]["base"], eps)
        if not raw["mlp"]:
            continue
        ff, mlp = slot(layer, "feed_forward"), raw["mlp"]
        if mlp["kind"] == "dense":
            assert (ff["kind"], ff["activation"], ff["gate_alpha"], ff["inner"], ff["gate_limit"]) == ("gated", "capped", 1.702, mlp["ff"], mlp["limit"])
        else:
            shared = mlp.get("shared", {}).get("ff", 0)
            assert (ff["kind"], ff["expert"], ff["activation"], ff["score"], ff["weight_on"]) == ("routed", "plain", "relu2", "softmax", "output") and ff["renormalise"]
            assert (ff["experts"], ff["top"], ff["inner"], ff["shared_inner"], ff["shared_gate"]) == (
                mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"], shared, shared > 0)


def test_absent_keys_have_their_obvious_meaning():
    c = copy.deepcopy(CONFIG_A)
    m = c["layers"][4]["mixer"]
    for k in ("kv_heads", "vdim", "scale", "softcap"):
        m.pop(k)
    for k in ("vdim", "scale"):
        c["layers"][2]["mixer"].pop(k)
    c.pop("embedding")
    d = describe_config(c)["spec"]
    a = slot(d["layers"][4], "mixer")
    assert (a["n_kv_head"], a["vdim"], a["soft_cap"]) == (5, 8, 0.0) and abs(a["scale"] - 8 ** -0.5) < 1e-12
    b = slot(d["layers"][2], "mixer")
    assert b["vdim"] == 4 and abs(b["scale"] - 12 ** -0.5) < 1e-12 and d["embedding"]["scale"] == 1.0


def test_checkpoint_map_names_the_files_tensors():
    d = describe_config(CONFIG_A)
    ck = d["checkpoint"]
    names = lambda path: [s["name"] for s in ck[path]["sources"]]
    assert names("layers.1.mixer.proj.weight") == ["l1.mix.q", "l1.mix.k", "l1.mix.v"] and names("layers.1.mixer.qkv_bias") == ["l1.mix.q.b", "l1.mix.k.b", "l1.mix.v.b"]
    assert names("layers.1.mixer.out.bias") == ["l1.mix.o.b"]
    assert names("layers.0.mixer.proj.weight") == ["l0.mix.dq", "l0.mix.dkv"] and names("layers.2.mixer.proj.weight") == ["l2.mix.dq", "l2.mix.dkv", "l2.mix.g"]
    assert names("layers.3.mixer.proj.weight") == ["l3.mix.dq"] and "layers.3.mixer.latent_norm.weight" not in ck
    assert names("layers.0.mixer_out_norm.weight") == ["l0.norm1b"] and names("layers.0.ff_out_norm.weight") == ["l0.norm2b"]
    assert names("layers.0.feed_forward.router.weight") == ["l0.mlp.router", "l0.mlp.shared.sg"] and names("layers.4.feed_forward.router.weight") == ["l4.mlp.router"]
    assert names("layers.0.feed_forward.experts.up.weight") == [f"l0.mlp.e{e}.up" for e in range(6)]
    assert names("layers.1.feed_forward.gate_up.weight") == ["l1.mlp.gate", "l1.mlp.up"]
    assert "layers.3.ff_norm.weight" not in ck and any("l3" in t and "norm2" in t for t in d["ignored_tensors"])


def test_weights_load_as_the_engine_holds_them(tmp_path):
    from liyab_b200.weights import load_parameters
    weights = random_weights(CONFIG_D, 3)
    path = write_model(str(tmp_path / "d"), CONFIG_D, weights)
    for dtype in ("float32", "bfloat16"):
        p = load_parameters(path, dtype)
        assert p["layers.0.feed_forward.router.weight"].shape == (2, 48)            # one expert, and the shared expert's gate
        assert p["layers.2.mixer.proj.weight"].shape == (1 + 3, 48) and p["layers.1.mixer.proj.weight"].shape == (1 + 3 + 1, 48)
        assert p["layers.3.mixer.qkv_bias"].shape == (2 * 16 + 16 + 1,) and p["layers.3.mixer.qkv_bias"].dtype == np.float32
        assert (p["layers.3.mixer.qkv_bias"][32:48] == np.float32(weights["l3.mix.k.b"])).all()
    # A tensor the design does not have is named in the refusal.
    weights["l1.mix.sink"] = weights["l0.mix.v.b"]
    with pytest.raises(LiyabError, match="l1.mix.sink"):
        load_parameters(write_model(str(tmp_path / "bad"), CONFIG_D, weights), "float32")


@pytest.mark.parametrize("edit, message", [
    (lambda c: c["layers"][0].update(type="retention"), "type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=0.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "scaling.fast"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0), "scaling.factor"),
    (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from"),          # an attention layer makes no latent rows
    (lambda c: c["layers"][5]["mixer"].update(kv_from=3), "kv_from"),          # that layer reads another's itself
    (lambda c: c["layers"][3]["mixer"].update(kv_rank=25), "kv_from"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(base=301.0), "kv_from"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "shared.ff"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gated"), "kind"),
    (lambda c: c["layers"][1]["mlp"].pop("limit"), "limit"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_refusals_name_the_key(edit, message):
    config = copy.deepcopy(CONFIG_A)
    edit(config)
    with pytest.raises(LiyabError, match=message):
        describe_config(config)


@pytest.mark.parametrize("dims, base, scaling", [(64, 5e5, (4.0, 2000, 32.0, 1.0)), (8, 100.0, (3.0, 64, 8.0, 0.5)), (2, 10.0, (2.0, 16, 2.0, 1.0)), (32, 1e4, (16.0, 4096, 1.0, 1.0)),
                                                 (128, 1e6, (1.5, 100, 1000.0, 0.001))])
def test_stretched_frequencies_by_counting_turns(dims, base, scaling):
    """The plain model's frequencies against what the stretching is for: a pair that turns often over the original length keeps its frequency, one that
    turns seldom has it divided, those between lie between and fall."""
    r = rotation(dims, base, scaling)
    f, magnitude = plain.frequencies(r)
    unscaled, one = plain.frequencies(rotation(dims, base))
    factor, original, fast, slow = scaling
    assert one == 1.0 and abs(magnitude - (1.0 + 0.1 * np.log(factor))) < 1e-12
    turns = original * unscaled / (2 * np.pi)
    step = base ** (2.0 / dims)                       # neighbouring pairs' ratio: the ends of the ramp are whole pairs, so they may lie one pair off
    ratio = f / unscaled
    assert (ratio <= 1 + 1e-12).all() and (ratio >= 1 / factor - 1e-12).all() and (np.diff(ratio) <= 1e-12).all()
    if max(fast, slow) < turns[0]:
        assert (ratio[turns > fast * step] == 1.0).all()
    assert np.allclose(ratio[(turns < slow / step) & (np.arange(dims // 2) > 0)], 1 / factor) or fast == slow


def test_cache_units_of_the_mixers():
    """Units side by side in one manager: grouped keys and values without a window, latent rows (one plane) without one and under one; a row that others read
    through a wider window stays as long as the widest reader sees it."""
    from liyab_b200.cache import CacheManager, KvNeed
    needs = {0: KvNeed(n_kv_head=1, head_dim=30, window=33, planes=1), 1: KvNeed(n_kv_head=2, head_dim=12, window=0), 2: KvNeed(n_kv_head=1, head_dim=48, window=0, planes=1)}
    cache = CacheManager(needs, {}, page_size=16, num_pages=16, max_requests=2)
    cache.open("a")
    cache.reserve("a", 100)
    cache.commit("a", 100)
    assert sorted(cache.pages_in_use().values()) == [3, 7, 7]        # the window of 33 keeps positions 68..99
    cache.close("a")
    assert sum(cache.pages_in_use().values()) == 0
    cache.check()
