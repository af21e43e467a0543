"""Mokisun's configuration, model description, checkpoint map and cache needs, and the plain model's own routing, without a GPU."""
from __future__ import annotations

import copy

import numpy as np
import pytest

import plain_mokisun as plain
from liyab_b200.config import describe_config, slot, supported_architectures
from liyab_b200.status import LiyabError
from mokisun_models import CONFIG_A, CONFIG_B, CONFIG_D, RANKS, random_weights, write_model


def test_registered_and_found_by_its_own_key():
    assert "mokisun" in supported_architectures()
    assert describe_config(CONFIG_A)["architecture"] == "mokisun"


def test_every_size_and_constant_comes_from_the_file():
    d = describe_config(CONFIG_A)["spec"]
    assert d["embedding"] == {"vocab_size": 150, "size": 96, "scale": 1.0} and d["streams"] == 3
    assert not d["head"]["tied"] and d["position"]["kind"] == "none" and d["final_norm"] == {"kind": "dynamic_tanh", "size": 96}
    assert [(e["layer"], e["cache"]) for e in d["run_order"]] == [(i, i) for i in range(6)]
    for layer, raw in zip(d["layers"], CONFIG_A["layers"]):
        assert layer["arrangement"] == "streams"
        names = [s["name"] for s in layer["slots"]]
        assert names == ["mixer_join", "mixer_norm", "mixer"] + (["ff_join", "ff_norm", "feed_forward"] if raw["mlp"] else [])
        assert slot(layer, "mixer_join") == {"kind": "hyper", "streams": 3, "size": 96, "layer_scale": True}
        assert slot(layer, "mixer_norm") == {"kind": "dynamic_tanh", "size": 96}
        m, r = slot(layer, "mixer"), raw["mixer"]
        if raw["type"] == "attention":
            assert m["kind"] == "gated_attention" and m["rot_layout"] == "interleaved" and m["sink"] and m["gate"] == "none" and not m["qk_norm"] and not m["bias"]
            assert (m["n_head"], m["n_kv_head"], m["dim"], m["vdim"], m["scale"], m["window"]) == (r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["scale"], r["mask"]["size"])
            assert (m["rot_dims"], m["rot_base"]) == (r["rot"]["dims"], r["rot"]["base"])
        elif raw["type"] == "gla":
            assert m["kind"] == "channel_memory" and m["rule"] == "linear" and m["decay"] == "sigmoid" and m["gate"] == "silu" and "taps" not in m
            assert (m["n_head"], m["dim"], m["vdim"], m["tau"], m["eps"]) == (r["heads"], r["dim"], r["vdim"], r["tau"], 1e-5)
            assert m["q_scale"] == pytest.approx(r["dim"] ** -0.5)
        else:
            assert m["kind"] == "branch_sum" and not m["norm"]
            left, right = m["branches"]
            assert (left["scale"], right["scale"]) == (r["left_scale"], r["right_scale"])
            l, rr = left["part"], right["part"]
            assert l["kind"] == "gated_attention" and l["values"] == "keys" and l["slopes"] and l["unit_sink"]
            assert (l["n_head"], l["n_kv_head"], l["dim"], l["scale"], l["window"]) == (r["left"]["heads"], r["left"]["kv_heads"], r["left"]["dim"], r["left"]["scale"],
                                                                                        r["left"]["mask"]["size"])
            assert rr["kind"] == "channel_memory" and rr["rule"] == "delta" and rr["decay"] == "softplus" and rr["unit"] and rr["gate"] == "sigmoid"
            assert (rr["n_head"], rr["n_kv_head"], rr["dim"], rr["vdim"], rr["taps"]) == tuple(r["right"][k] for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
        if raw["mlp"]:
            ff, router = slot(layer, "feed_forward"), raw["mlp"]["router"]
            assert ff["kind"] == "routed" and ff["score"] == "softmax" and not ff["renormalise"] and ff["correction"] and ff["weight_on"] == "output"
            assert (ff["experts"], ff["identity"], ff["top"], ff["inner"], ff["groups"], ff["keep_groups"], ff["route_scale"]) == (
                router["experts"], router["identity"], router["top"], raw["mlp"]["expert"]["ff"], router["groups"]["count"], router["groups"]["keep"], router["scale"])


def test_checkpoint_map_names_the_files_tensors():
    d = describe_config(CONFIG_A)
    ck = d["checkpoint"]
    names = lambda path: [s["name"] for s in ck[path]["sources"]]
    assert names("layers.0.mixer.proj.weight") == [f"l0.mix.{x}" for x in ("q", "k", "v", "a1", "g")]
    assert names("layers.1.mixer.proj.weight") == ["l1.mix.q", "l1.mix.k", "l1.mix.v"]
    assert names("layers.2.mixer.left.proj.weight") == ["l2.mix.left.q", "l2.mix.left.k"]
    assert names("layers.2.mixer.right.proj.weight") == [f"l2.mix.right.{x}" for x in ("q", "k", "v", "a1", "g1", "b")]
    assert names("layers.2.mixer.right.conv.weight") == [f"l2.mix.right.{x}.conv" for x in "qkv"] and ck["layers.2.mixer.right.conv.weight"]["kind"] == "vector"
    assert names("layers.2.mixer_join.mix") == ["l2.hc1.mix"] and names("layers.2.ff_join.scale") == ["l2.ls2"]
    assert names("layers.0.mixer_norm.alpha") == ["l0.norm1.alpha"] and ck["layers.0.mixer_norm.alpha"]["repeat"] == 1
    assert names("layers.0.feed_forward.router.correction") == ["l0.mlp.correction"]
    assert len(names("layers.0.feed_forward.experts.gate_up.weight")) == 12        # the identities have no matrices
    assert "layers.3.ff_norm.weight" not in ck and any("l3" in t and "norm2" in t for t in d["ignored_tensors"])


def test_ranks_come_from_the_files_shapes(tmp_path):
    from liyab_b200.weights import load_parameters
    for name, config in (("A", CONFIG_A), ("D", CONFIG_D)):
        r1, r2 = RANKS[name]
        path = write_model(str(tmp_path / name), config, random_weights(config, 3, RANKS[name]))
        for dtype in ("float32", "bfloat16"):
            p = load_parameters(path, dtype)
            g, right = (0, 2) if name == "A" else (0, 1)
            m = config["layers"][g]["mixer"]
            assert p[f"layers.{g}.mixer.decay.weight"].shape == (m["heads"] * m["dim"], r1)
            r = config["layers"][right]["mixer"]["right"]
            assert p[f"layers.{right}.mixer.right.gate.weight"].shape == (r["heads"] * r["vdim"], r2)
            assert p[f"layers.{right}.mixer.right.conv.weight"].dtype == np.float32 and p[f"layers.{right}.mixer_norm.alpha"].shape == (1,)
    # A tensor the design does not have, or one of another shape, is named in the refusal.
    weights = random_weights(CONFIG_D, 3, (1, 1))
    weights["l0.mix.sink"] = np.zeros(1)
    with pytest.raises(LiyabError, match="l0.mix.sink"):
        load_parameters(write_model(str(tmp_path / "bad"), CONFIG_D, weights), "float32")
    weights = random_weights(CONFIG_D, 3, (1, 1))
    weights["l0.mix.a2"] = np.zeros((1, 3))
    with pytest.raises(LiyabError, match="l0.mix.a2"):
        load_parameters(write_model(str(tmp_path / "bad2"), CONFIG_D, weights), "float32")


def test_random_weights_mode_writes_what_it_can_read(tmp_path):
    from liyab_b200.weights import load_parameters, write_random_model
    config = copy.deepcopy(CONFIG_B)
    config["layers"][2]["mixer"]["a_rank"] = 11
    path = write_random_model(str(tmp_path / "r"), config, seed=4, dtype="bfloat16")
    p = load_parameters(path, "bfloat16")
    assert p["layers.2.mixer.decay.weight"].shape == (4 * 64, 11)


@pytest.mark.parametrize("edit, message", [
    (lambda c: c["layers"][0].update(type="retention"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("tau"), "tau"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["left"].update(vdim=13), "left.vdim"),
    (lambda c: c["layers"][2]["mixer"]["right"].pop("conv"), "right.conv"),
    (lambda c: c["layers"][2]["mixer"]["right"].update(kv_heads=3), "right.kv_heads"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3), "groups.count"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=5), "groups.keep"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_refusals_name_the_key(edit, message):
    config = copy.deepcopy(CONFIG_A)
    edit(config)
    with pytest.raises(LiyabError, match=message):
        describe_config(config)


def test_the_plain_routing():
    """Groups by their best choice score, corrections in the choice only, hidden experts at minus infinity (negative choice scores stay eligible)."""
    s = np.array([0.30, 0.05, 0.25, 0.20, 0.15, 0.05])
    router = dict(experts=5, top=2, identity=1, scale=1.0, groups=dict(count=3, keep=2))
    assert plain.choose(s, np.zeros(6), router).tolist() == [0, 2]
    assert plain.choose(s, np.full(6, -2.0), router).tolist() == [0, 2]
    assert plain.choose(s, np.array([0, 0, -0.5, -0.5, 0, 0]), router).tolist() == [0, 4]
    assert plain.choose(s, np.array([-1.0, -1.0, -1.0, -1.0, -0.8, -2.0]), router).tolist() == [4, 0]
    assert plain.choose(s, np.zeros(6), dict(router, groups=dict(count=3, keep=1))).tolist() == [0, 1]
