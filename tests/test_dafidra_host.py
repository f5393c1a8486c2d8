"""Dafidra without a GPU: configuration reader, the oracle's own consistency, and that the GPU tests' inputs would show a fault."""
import copy

import numpy as np
import pytest

import dafidra_models as M
from oracle import dafidra_ref as D


def test_config_reader_accepts_the_shapes_and_reports_the_base_configuration(R):
    for cfg in (M.ODD, M.WIDE, M.BROAD, M.LAST_MIXER):
        c = R.config_info(cfg)
        a = cfg["layers"][0]["mixer"]["left"]
        assert (c.dim, c.vocab, c.nlayers) == (cfg["width"], cfg["vocab"], len(cfg["layers"]))
        assert (c.heads, c.kv_heads, c.hd) == (a["heads"], a["kv_heads"], a["dim"])


@pytest.mark.parametrize("change,message", [
    (lambda c: c.update(architecture="Unheard"), "unknown architecture"),
    (lambda c: c.pop("architecture"), "names no architecture"),
    (lambda c: c.pop("width"), 'missing "width"'),
    (lambda c: c.update(vocab=3.5), "positive integer"),
    (lambda c: c.update(layers=[]), "non-empty list"),
    (lambda c: c["layers"][0].update(type="serial"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), 'missing "right"'),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "unknown kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=13), "exceeds the experts"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5), "groups must divide"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=0), "gate_cap must be positive"),
])
def test_config_reader_names_what_is_wrong(R, change, message):
    cfg = copy.deepcopy(M.ODD)
    change(cfg)
    with pytest.raises(ValueError, match=message):
        R.config_info(cfg)


def test_config_text_that_is_not_an_object(R):
    for text in ("", "[]", '{"architecture": "Dafidra", ', "nonsense"):
        with pytest.raises(ValueError):
            R.config_info(text)


def test_oracle_memory_is_the_same_token_by_token_and_from_a_carried_state():
    cfg, W = M.ODD, M.f64(M.weights(M.ODD, 3))
    c = cfg["layers"][0]["mixer"]["right"]
    h = np.random.default_rng(0).standard_normal((40, cfg["width"]))
    whole = D.matrix_memory(h, W, "l0.mix.right.", c, 1e-5)
    state = (np.zeros((c["heads"], c["dim"], c["vdim"])), np.zeros((c["heads"], c["dim"])), np.zeros(c["heads"]))
    parts = np.concatenate([D.matrix_memory(h[a:b], W, "l0.mix.right.", c, 1e-5, state=state) for a, b in ((0, 1), (1, 17), (17, 40))])
    assert np.abs(whole - parts).max() < 1e-12


def test_oracle_window_of_one_sees_only_itself_and_the_sink():
    """With a window of one position the softmax is v / (1 + exp(sink - score)): a closed form without the loop."""
    cfg = M.config(32, 50, [(M.attn(2, 1, 8, 8, 1, 0.7), M.memory(1, 8, 8, 5.0), None)])
    W = M.f64(M.weights(cfg, 5))
    h, p, a = np.random.default_rng(1).standard_normal((5, 32)), "l0.mix.left.", cfg["layers"][0]["mixer"]["left"]
    q = D.norm_plain(h @ W[p + "q"].T, W[p + "q.norm"], 1e-5) * D.query_temperature(np.arange(5), 7, 0.4)[:, None]
    k, v = D.norm_plain(h @ W[p + "k"].T, W[p + "k.norm"], 1e-5), h @ W[p + "v"].T
    s = np.stack([(q[:, i * 8:i * 8 + 8] * k).sum(1) * 0.7 for i in range(2)], 1)
    w = 1 / (1 + np.exp(W[p + "sink"] - s)) * D.sigmoid(h @ W[p + "g"].T)
    want = np.concatenate([w[:, i:i + 1] * v for i in range(2)], 1) @ W[p + "o"].T
    assert np.abs(D.attention(h, W, p, a, 1e-5) - want).max() < 1e-12


def test_oracle_routing_respects_groups_and_keeps_the_scores():
    z = np.log(np.array([.30, .02, .01, .01, .20, .18, .04, .04, .10, .10]))
    ids, w = D.route(z, 10, 3, {"count": 5, "keep": 2})       # groups of two: bests .30 .01 .20 .04 .10
    assert ids.tolist() == [0, 4, 5] and np.allclose(w, [.30, .20, .18])
    ids, _ = D.route(z, 10, 3, {"count": 5, "keep": 1}, fault="no_groups")
    assert ids.tolist() == [0, 4, 5]
    ids, _ = D.route(z, 10, 2, {"count": 5, "keep": 1})
    assert ids.tolist() == [0, 1]


@pytest.mark.parametrize("fault", ["norm_per_head", "no_temperature", "window_plus", "window_minus", "no_bias", "no_sink", "no_gate", "no_groups"])
def test_the_random_models_show_a_fault_of_each_mechanism(fault):
    """A mistake in one mechanism moves the logits far beyond what the GPU tests accept."""
    W = M.f64(M.weights(M.ODD, 2))
    ids = np.random.default_rng(2).integers(0, M.ODD["vocab"], 60)
    assert M.error(D.forward(M.ODD, W, ids, fault=fault), D.forward(M.ODD, W, ids)) > 0.1


def test_the_pointed_query_shows_one_key_more_or_less():
    cfg, W, ids, places = M.window_case(11)
    W64 = M.f64(W)
    ref = D.forward(cfg, W64, ids)
    for fault in ("window_plus", "window_minus"):
        bad = D.forward(cfg, W64, ids, fault=fault)
        hit = places["out" if fault == "window_plus" else "in"]
        assert min(M.error(bad[p], ref[p]) for p in hit) > 0.1
