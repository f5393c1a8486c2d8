"""Kazodra without a GPU: configuration reader, the oracle's own consistency, and that the GPU tests' inputs would show a fault."""
import copy

import numpy as np
import pytest

import kazodra_models as M
from oracle import kazodra_ref as K


def test_config_reader_accepts_the_shapes_and_reports_the_base_configuration(R):
    for cfg in (M.ODD, M.WIDE, M.BROAD, M.PLAIN, M.TAIL):
        c = R.config_info(cfg)
        assert (c.dim, c.vocab, c.nlayers, c.heads) == (cfg["width"], cfg["vocab"], len(cfg["layers"]), cfg["layers"][0]["mixer"]["heads"])


def set_mixer(i, **kw):
    return lambda c: c["layers"][i]["mixer"].update(kw)


@pytest.mark.parametrize("change,message", [
    (lambda c: c.pop("width"), 'missing "width"'),
    (lambda c: c.pop("norm"), 'missing "norm"'),
    (lambda c: c["layers"][0].update(type="parallel"), "unknown mixer type"),
    (lambda c: c["layers"][0].pop("mixer"), 'missing "mixer"'),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe", expert={"ff": 8}, router={"experts": 4, "top": 2}), "must be dense"),
    (set_mixer(0, kv_heads=4), "multiple of kv_heads"),
    (set_mixer(0, rot={"dims": 7, "base": 10.0}), "even"),
    (set_mixer(0, rot={"dims": 14, "base": 10.0}), "no more than"),
    (set_mixer(0, rot={"dims": 8, "base": 0}), "base must be positive"),
    (set_mixer(0, rot={"dims": 8, "base": 10.0, "scaling": {"factor": 2.0, "low": 1.0, "high": 4.0}}), 'missing "original"'),
    (set_mixer(0, diff=None), 'missing "diff"'),
    (set_mixer(1, kv_rank=0), "positive integer"),
    (set_mixer(2, decay=[0.5, 0.5]), "one number per head"),
    (set_mixer(2, decay=[0.5, 1.5, 0.2]), "between 0 and 1"),
    (set_mixer(2, decay=0.5), "must be a list"),
    (lambda c: c["loop"].update(stop=6), "run of the layers"),
    (lambda c: c["loop"].update(start=4), "run of the layers"),
    (lambda c: c["loop"].update(start=-1), "non-negative"),
    (lambda c: c["token_side"].update(dim=0), "positive integer"),
])
def test_config_reader_names_what_is_wrong(R, change, message):
    cfg = copy.deepcopy(M.ODD)
    change(cfg)
    with pytest.raises(ValueError, match=message):
        R.config_info(cfg)


def test_optional_parts_may_be_null(R):
    cfg = copy.deepcopy(M.PLAIN)
    cfg["loop"] = cfg["token_side"] = None
    assert R.config_info(cfg).nlayers == 3


def test_the_models_cover_the_frequency_bands():
    """Kept, blended and stretched wavelengths all occur, and the blend meets both ends."""
    r = M.ODD["layers"][0]["mixer"]["rot"]
    base = {k: v for k, v in r.items() if k != "scaling"}
    q = K.frequencies(r) / K.frequencies(base)
    assert q[0] == 1.0 and np.isclose(q[-1], 0.25) and any(0.25 < x < 1.0 for x in q[1:-1])


def test_rotation_keeps_products_at_a_distance_and_leaves_the_rest():
    rng = np.random.default_rng(0)
    r, pos = M.rot(6, 50.0), np.array([3.0, 10.0, 40.0, 47.0])
    q, k = np.tile(rng.standard_normal(8), (4, 1)), np.tile(rng.standard_normal(8), (4, 1))
    a, b = K.rotate(q, pos, r), K.rotate(k, pos, r)
    assert np.isclose(a[1] @ b[0], a[3] @ b[2]) and not np.isclose(a[1] @ b[0], a[0] @ b[0])
    assert np.array_equal(a[:, 6:], q[:, 6:]) and np.allclose(a[0, 0], q[0, 0] * np.cos(3.0) - q[0, 1] * np.sin(3.0))


def test_oracle_linear_attention_carries_its_state():
    cfg, W = M.ODD, M.f64(M.weights(M.ODD, 3))
    c = cfg["layers"][2]["mixer"]
    h = np.random.default_rng(0).standard_normal((40, cfg["width"]))
    whole = K.lightning(h, W, "l2.mix.", c, 1e-5)
    state = np.zeros((c["heads"], c["dim"], c["vdim"]))
    parts = np.concatenate([K.lightning(h[a:b], W, "l2.mix.", c, 1e-5, state=state) for a, b in ((0, 1), (1, 17), (17, 40))])
    assert np.abs(whole - parts).max() < 1e-12


def test_oracle_latent_attention_in_absorbed_form():
    """Scores as the query carried into the latent space, values after the weighted sum: the same numbers."""
    cfg, W = M.ODD, M.f64(M.weights(M.ODD, 3))
    c, p = cfg["layers"][1]["mixer"], "l1.mix."
    H, nd, rd, vd, R = (c[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    h = np.random.default_rng(0).standard_normal((20, cfg["width"]))
    pos = np.arange(20.0)
    q, low = (h @ W[p + "q"].T).reshape(20, H, nd + rd), h @ W[p + "dkv"].T
    lat = K.rms(low[:, :R], 1e-5) * W[p + "dkv.norm"]
    kr, qr = K.rotate(low[:, R:], pos, c["rot"]), K.rotate(q[..., nd:], pos, c["rot"])
    out = np.zeros((20, H, vd))
    for a in range(H):
        s = (q[:, a, :nd] @ W[p + "uk"][a * nd:(a + 1) * nd]) @ lat.T + qr[:, a] @ kr.T
        out[:, a] = K.softmax_rows(s * c["scale"], K.visible(20, c["mask"]["size"])) @ lat @ W[p + "uv"][a * vd:(a + 1) * vd].T
    assert np.abs(out.reshape(20, -1) @ W[p + "o"].T - K.latent_attention(h, W, p, c, 1e-5)).max() < 1e-10


def test_oracle_order_of_the_layer_runs():
    assert K.layer_runs(M.ODD) == [(0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None), (1, 2), (2, None), (3, None), (4, None)]
    assert K.layer_runs(M.TAIL) == [(0, None), (1, 0), (2, None)]


@pytest.mark.parametrize("fault", ["norm_keeps_mean", "norm_no_bias", "no_scaling", "half_layout", "window_plus", "window_minus", "no_latent_norm", "shared_key_unrotated",
                                   "no_rotated_part", "one_map", "heads_interleaved", "no_head_norm", "no_gate", "decay_after", "no_decay", "norm_per_head", "first_part",
                                   "no_side", "one_pass", "no_step", "first_step"])
def test_the_random_models_show_a_fault_of_each_mechanism(fault):
    """A mistake in one mechanism moves the logits far beyond what the GPU tests accept."""
    W = M.f64(M.weights(M.ODD, 2))
    ids = np.random.default_rng(2).integers(0, M.ODD["vocab"], 60)
    assert M.error(K.forward(M.ODD, W, ids, fault=fault), K.forward(M.ODD, W, ids)) > 0.1


def test_the_pointed_query_shows_one_key_more_or_less():
    cfg, W, ids, places = M.edge_case(11)
    W64 = M.f64(W)
    ref = K.forward(cfg, W64, ids)
    for fault in ("window_plus", "window_minus"):
        bad = K.forward(cfg, W64, ids, fault=fault)
        hit = places["out" if fault == "window_plus" else "in"]
        assert min(M.error(bad[p], ref[p]) for p in hit) > 0.1
