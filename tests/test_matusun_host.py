"""Matusun without a device: the configuration (every key, absent keys, wrong values), the manifest against the tensor
names of a checkpoint, the run order of repeated layers, and the plain implementation's parts on cases that can be
worked out by hand."""
import math

import numpy as np
import pytest

import matusun_tools as mt
import plain_matusun as P
from gollmgo_b200.config import ConfigError, resolve_architecture
from gollmgo_b200.config.matusun_config import MatusunConfig, RowNormedAttentionConfig, SelectiveScanConfig
from gollmgo_b200.parts import looped_run_order
from gollmgo_b200.parts.model import manifest_for_config


@pytest.mark.parametrize("name", sorted(mt.TINY))
def test_manifest_is_the_checkpoint(name):
    cfg, _ = mt.get(name)
    got = {k: tuple(v.shape) for k, v in manifest_for_config(cfg).items() if not v.optional}
    assert got == mt.tensor_shapes(cfg)


def test_every_key_is_read():
    cfg, _ = mt.get("mat_a")
    c = MatusunConfig.from_dict(cfg)
    assert (c.vocab, c.width, c.eps, c.streams, len(c.layers)) == (203, 64, 1e-5, 2, 4)
    assert (c.loop.start, c.loop.stop, c.loop.times) == (1, 3, 2)
    s, a = c.layers[0].mixer, c.layers[1].mixer
    assert isinstance(s, SelectiveScanConfig) and isinstance(a, RowNormedAttentionConfig)
    assert (s.inner, s.state, s.dt_rank, s.conv) == (96, 8, 5, 4)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.rot) == (4, 2, 32, 16, 0.3, 20, (10000.0, 20))
    f = c.layers[0].mlp
    assert (f.ff, f.experts, f.top, f.identity, f.scale, f.shared_ff) == (40, 5, 2, 2, 1.5, 24)


def test_absent_keys_switch_their_feature_off():
    cfg, _ = mt.get("mat_a")
    c = MatusunConfig.from_dict(cfg)
    spec = resolve_architecture(cfg).spec(c)
    assert c.layers[3].mixer.window is None and spec.layers[3].mixer["position"].kind == "none"
    assert c.layers[2].mlp is None and spec.layers[2].feed_forward is None and spec.layers[2].ffn_norm is None
    assert c.layers[3].mlp.shared_ff is None and c.layers[3].mlp.scale == 1.0 and c.layers[1].mlp.identity == 0
    cfg, _ = mt.get("mat_b")
    assert MatusunConfig.from_dict(cfg).loop is None


@pytest.mark.parametrize("name,order", [("mat_a", [0, 1, 2, 1, 2, 3]), ("mat_b", [0, 1, 2]), ("mat_c", [0, 1, 0, 1, 0, 1, 2, 3]),
                                        ("mat_d", [0, 1, 2, 0, 1, 2]), ("mat_e", [0, 1, 1, 1, 2])])
def test_repeated_layers_have_a_cache_per_pass(name, order):
    cfg, _ = mt.get(name)
    spec = resolve_architecture(cfg).spec(MatusunConfig.from_dict(cfg))
    assert [e.layer for e in spec.run_order] == order == P.passes(cfg)
    assert [e.cache for e in spec.run_order] == list(range(len(order)))
    assert all(e.writes_cache and not e.mix_input for e in spec.run_order)
    assert len(spec.layers) == len(cfg["layers"])


def test_run_order_that_mixes_the_input_in():
    runs = looped_run_order(4, 1, 3, 2, mix_input=True)
    assert [(e.layer, e.cache, e.mix_input) for e in runs] == [(0, 0, False), (1, 1, True), (2, 2, False), (1, 3, True), (2, 4, False),
                                                               (3, 5, False)]


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][1].update(type="conv"), "type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=34), "at most"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(base=0), "base"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "positive"),
    (lambda c: c["layers"][0]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "picks"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "known"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_wrong_values_are_refused(change, message):
    cfg, _ = mt.get("mat_a")
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        MatusunConfig.from_dict(cfg)


def test_plain_streams_by_hand():
    x = np.array([[[1.0]], [[10.0]]])
    assert P.contract(x, np.array([0.5, 2.0])).tolist() == [[20.5]]
    mix = np.array([[1.0, 2.0], [3.0, 4.0]])               # [from, to]
    assert P.spread(x, mix, np.array([1.0, -1.0]), np.array([[100.0]])).tolist() == [[[131.0]], [[-58.0]]]


def test_plain_scan_by_hand():
    # one channel, one state: S_1 = dt x B, S_2 = exp(dt A) S_1 + dt x B
    one = np.ones((2, 1))
    y = P.selective_scan(one * [[2.0], [3.0]], one * 0.5, np.array([[-1.0]]), one * 4.0, one, np.array([10.0]))
    assert np.allclose(y[:, 0], [4.0 + 20.0, 4.0 * math.exp(-0.5) + 6.0 + 30.0])
    # the last column of the taps is the current token's
    assert P.causal_conv(np.array([[1.0], [5.0]]), np.array([[2.0, 3.0]]), np.array([0.5])).tolist() == [[3.5], [17.5]]


def test_plain_router_by_hand():
    w = np.log(np.array([[0.1], [0.2], [0.3], [0.4]]))
    r = {"top": 2, "scale": 3.0}
    idx, wgt = P.route(np.ones((1, 1)), w, np.zeros(4), r)
    assert idx.tolist() == [[3, 2]] and np.allclose(wgt, [[3 * 4 / 7, 3 * 3 / 7]])
    idx, wgt = P.route(np.ones((1, 1)), w, np.array([0.5, 0.0, 0.0, 0.0]), r)       # the choice moves, the weights do not
    assert idx.tolist() == [[0, 3]] and np.allclose(wgt, [[3 * 1 / 5, 3 * 4 / 5]])
    # an identity expert hands its input on
    f = {"router": {"experts": 1, "identity": 1, "top": 1, "scale": 2.0}}
    h = np.array([[1.5]])
    w = {"p.router": np.array([[0.0], [9.0]]), "p.correction": np.zeros(2), "p.e0.up": np.ones((1, 1)), "p.e0.down": np.ones((1, 1))}
    assert np.allclose(P.mixture(h, w, "p.", f), 2.0 * h)
    w["p.router"] = w["p.router"][::-1]
    assert np.allclose(P.mixture(h, w, "p.", f), 2.0 * 1.5 ** 2)


def test_plain_norm_is_over_all_heads():
    h, I = np.array([[3.0, 4.0]]), np.eye(2)
    w = {"p.q": I, "p.k": I, "p.v": I, "p.o": I, "p.q.norm": np.ones(2), "p.k.norm": np.ones(2)}
    m = {"heads": 2, "kv_heads": 2, "dim": 1, "vdim": 1, "scale": 1.0}
    x = np.concatenate([h, 2 * h])
    y = P.attention(x, w, "p.", m, 0.0)
    q = h[0] / math.sqrt(12.5)                              # both rows have this direction
    for hd in range(2):
        assert np.isclose(y[1, hd], 1.5 * h[0, hd]) and np.isclose(q[hd] ** 2, h[0, hd] ** 2 / 12.5)
