"""Rimidra without a device: the configuration (every key, absent keys, wrong values), the manifest against the
tensor names of a checkpoint, layers that use another layer's weights, and the plain implementation's parts on
cases that can be worked out by hand."""
import math

import numpy as np
import pytest

import plain_rimidra as P
import rimidra_tools as rt
from gollmgo_b200.config import ConfigError, resolve_architecture
from gollmgo_b200.config.rimidra_config import RetentionConfig, RimidraConfig, SlopedAttentionConfig
from gollmgo_b200.parts.model import manifest_for_config
from gollmgo_b200.parts.position import inverse_frequencies


@pytest.mark.parametrize("name", sorted(rt.TINY))
def test_manifest_is_the_checkpoint(name):
    cfg, _ = rt.get(name)
    assert {k: tuple(v.shape) for k, v in manifest_for_config(cfg).items()} == rt.tensor_shapes(cfg)


def test_every_key_is_read():
    cfg, _ = rt.get("rim_a")
    c = RimidraConfig.from_dict(cfg)
    assert (c.vocab, c.width, c.eps, len(c.layers)) == (203, 64, 1e-5, 5)
    ret, att = c.layers[0].mixer, c.layers[1].mixer
    assert isinstance(ret, RetentionConfig) and isinstance(att, SlopedAttentionConfig)
    assert (ret.heads, ret.dim, ret.vdim, ret.decay, ret.rot) == (3, 16, 24, (0.9, 0.97, 0.995), (10000.0, 8))
    assert (att.heads, att.kv_heads, att.dim, att.vdim, att.scale, att.window, att.q_temp) == (4, 2, 32, 16, 0.3, 20, (0.7, 16.0))
    f = c.layers[0].mlp
    assert (f.kind, f.ff, f.experts, f.top, f.shared_ff) == ("moe", 40, 5, 2, 24)
    assert (c.layers[1].mlp.kind, c.layers[1].mlp.ff) == ("dense", 48) and c.layers[2].mlp is None
    assert [l.weights_of for l in c.layers] == [None, None, None, 0, 1]


def test_absent_keys_switch_their_feature_off():
    cfg, _ = rt.get("rim_a")
    c = RimidraConfig.from_dict(cfg)
    assert c.layers[2].mixer.window is None and c.layers[2].mixer.q_temp is None
    cfg, _ = rt.get("rim_c")
    c = RimidraConfig.from_dict(cfg)
    spec = resolve_architecture(cfg).spec(c)
    assert c.layers[3].mixer.rot is None and spec.layers[3].mixer["position"].kind == "none"
    assert c.layers[3].mlp.shared_ff is None and not spec.layers[3].feed_forward["shared_gate"]
    assert spec.layers[1].feed_forward is None


@pytest.mark.parametrize("name,owners", [("rim_a", [0, 1, 2, 0, 1]), ("rim_b", [1, 0, 1, 2]), ("rim_d", [0, 1, 2, 0, 3])])
def test_a_layer_with_anothers_weights_is_a_run_of_it_with_its_own_cache(name, owners):
    cfg, _ = rt.get(name)
    spec = resolve_architecture(cfg).spec(RimidraConfig.from_dict(cfg))
    assert [e.layer for e in spec.run_order] == owners
    assert [e.cache for e in spec.run_order] == list(range(len(owners))) and all(e.writes_cache for e in spec.run_order)
    assert len(spec.layers) == len(set(owners))
    named = [i for i, l in enumerate(cfg["layers"]) if l.get("weights_of") is None]
    assert [l.mixer_prefix for l in spec.layers] == [f"l{i}.mix." for i in named]


def test_a_chain_of_owners_ends_at_the_layer_with_tensors():
    cfg, _ = rt.get("rim_a")
    cfg["layers"][4] = dict(cfg["layers"][3], weights_of=3)
    c = RimidraConfig.from_dict(cfg)
    assert [l.weights_of for l in c.layers] == [None, None, None, 0, 0]


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][1].update(type="conv"), "type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "at most"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.9, 0.9]), "decay"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.9, 0.9, 1.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "positive"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "picks"),
    (lambda c: c["layers"][0]["mlp"].update(kind="mlp"), "known"),
    (lambda c: c["layers"][3].update(weights_of=9), "weights_of"),
    (lambda c: c["layers"][0].update(weights_of=3), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=1), "differs"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_wrong_values_are_refused(change, message):
    cfg, _ = rt.get("rim_a")
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        RimidraConfig.from_dict(cfg)


def test_rotation_table_is_the_plain_one():
    f = inverse_frequencies(12, 700.0, None).numpy()
    x = np.zeros((4, 1, 16))
    x[:, 0, 2], x[:, 0, 13] = 1.0, 5.0
    y = P.rotate_halves(x, {"dims": 12, "base": 700.0})
    for p in range(4):
        assert abs(y[p, 0, 2] - math.cos(p * f[2])) < 1e-12 and abs(y[p, 0, 8] - math.sin(p * f[2])) < 1e-12
        assert y[p, 0, 13] == 5.0


def test_plain_parts_by_hand():
    assert P.distance_slopes(4).tolist() == [0.25, 0.0625, 0.015625, 0.00390625]
    t = P.query_temperature(np.arange(8), {"coef": 0.5, "every": 4})
    assert np.allclose(t, [1, 1, 1, 1 + 0.5 * math.log(2)] + [1 + 0.5 * math.log(2)] * 3 + [1 + 0.5 * math.log(3)])
    seen = P.visible_keys(6, 3)
    assert seen[5].tolist() == [False, False, False, True, True, True] and seen[1].tolist() == [True, True] + [False] * 4
    pr = P.sink_softmax(np.zeros((1, 2)), np.array([[True, False]]), 0.0)
    assert pr.tolist() == [[0.5, 0.0]]
    assert P.choose(np.array([[0.2, 0.9, 0.9, 0.1]]), 2).tolist() == [[1, 2]]
    # retention of one head with d = dv = 1, no rotation: a leaky sum
    w = {"p." + k: np.ones((1, 1)) for k in ("q", "k", "v", "o")}
    w["p.g"] = np.array([[1.0]])
    h = np.array([[1.0], [2.0]])
    o = P.retention(h, w, "p.", {"heads": 1, "dim": 1, "vdim": 1, "decay": [0.5]}, 0.0)
    assert np.allclose(o, P.silu(h))                        # one value: divided by its own size it is 1
