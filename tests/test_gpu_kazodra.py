"""The Kazodra decoder on the GPU against its plain restatement (oracle/kazodra_ref.py): each mechanism alone, whole models,
prompt passes against token-by-token decoding, portions, window edges, far keys, rewinding, generation, the trace runner."""
import copy
import json
import os
import subprocess

import numpy as np
import pytest

import kazodra_models as M
from oracle import kazodra_ref as K

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# fp32: summation order only.  bf16 weights (exact in both): fp16 cache rows and 16 + 16 bit GEMM operands; KEPT is the
# distance to an oracle whose cache rounds its rows the same way.
TOL = {"f32": 4e-5, "bf16": 1.5e-2}
KEPT = {"decoded": 1e-3, "prompt": 6e-3}   # a prompt rounds the expanded keys and values of latent attention once more
SEED = {"ODD": 2, "WIDE": 5, "BROAD": 1, "PLAIN": 1, "TAIL": 3, "RAGGED": 4}


@pytest.fixture(scope="module")
def made(tmp_path_factory):
    """(configuration, weights, folder, tokens, oracle logits) by name, made once."""
    cache = {}

    def get(name, n=200):
        if name not in cache:
            cfg, seed = getattr(M, name), SEED[name]
            W = M.weights(cfg, seed)
            path = M.write_folder(tmp_path_factory.mktemp(name) / "m", cfg, W)
            ids = np.random.default_rng(seed).integers(0, cfg["vocab"], n)
            cache[name] = cfg, W, path, ids, K.forward(cfg, M.f64(W), ids)
        return cache[name]

    return get


def folder(tmp_path, cfg, W):
    return M.write_folder(tmp_path / "model", cfg, W)


def all_logits(m, ids, portion=None):
    """Logits at every token, fed in portions (a number, a list of sizes, or all at once)."""
    ids, out, at = list(ids), [], 0
    sizes = portion if isinstance(portion, list) else [portion or len(ids)] * len(ids)
    for n in sizes:
        part = ids[at:at + n]
        if not part:
            break
        out.append(m.prefill_logits(part, list(range(len(part)))))
        at += len(part)
    assert at == len(ids)
    return np.concatenate(out)


# ---------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(SEED))
def test_whole_prompt_and_decoding_match_the_oracle(R, made, name, dtype):
    cfg, W, path, ids, ref = made(name)
    m = R.Model.from_pretrained(path, max_tokens=256, dtype=dtype, page_tokens=16)
    got = all_logits(m, ids)
    m.set_len(0)
    one = np.stack([m.decode_token_logits_from_id(int(t)) for t in ids])
    print(name, dtype, "to the oracle:", M.error(got, ref), M.error(one, ref))
    assert M.error(got, ref) < TOL[dtype]
    assert M.error(one, ref) < TOL[dtype]
    if dtype == "bf16":
        rounded = K.forward(cfg, M.f64(W), ids, cache=np.float16)
        print("with rounded cache rows:", M.error(got, rounded), M.error(one, rounded))
        assert M.error(got, rounded) < KEPT["prompt"] and M.error(one, rounded) < KEPT["decoded"]


@pytest.mark.parametrize("name,portions", [
    ("ODD", [2] * 100), ("ODD", [9, 2, 13, 8, 64, 3, 65, 2, 34]), ("WIDE", [63, 2, 64, 1, 65, 5]), ("PLAIN", [8] * 25), ("BROAD", [130, 3, 50, 2, 15]), ("TAIL", [2, 11, 100, 1, 86]),
    ("RAGGED", [50, 2, 9, 1, 138]),
])
def test_portions_of_a_prompt_do_not_change_its_logits(R, made, name, portions):
    cfg, _, path, ids, ref = made(name)
    m = R.Model.from_pretrained(path, max_tokens=200, page_tokens=32, use_graph=True)
    assert M.error(all_logits(m, ids, list(portions)), ref) < TOL["bf16"]


@pytest.mark.parametrize("name", ["ODD", "WIDE"])
def test_long_prompts_are_processed_in_pieces(R, made, monkeypatch, name):
    cfg, _, path, ids, ref = made(name)
    monkeypatch.setenv("CD_PREFILL_ROWS", "70")
    m = R.Model.from_pretrained(path, max_tokens=200)
    assert M.error(all_logits(m, ids), ref) < TOL["bf16"]


def test_bf16_cache_and_single_rounding_options(R, made, monkeypatch):
    cfg, _, path, ids, ref = made("WIDE")
    m = R.Model.from_pretrained(path, max_tokens=200, kv_dtype="bf16")
    assert M.error(all_logits(m, ids, [150, 2, 48]), ref) < 4e-2
    monkeypatch.setenv("CD_PREFILL", "fast")
    m.set_len(0)
    assert M.error(all_logits(m, ids), ref) < 8e-2


# ---------------------------------------------------------------------- each mechanism alone
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("layer,part", [(0, "mix"), (0, "mlp"), (0, "side"), (1, "mix"), (2, "mix"), (3, "mix"), (4, "mix"), (4, "side")])
def test_each_mechanism_alone(R, tmp_path, layer, part, dtype):
    """One layer of ODD with its other sublayers neutral: the hidden state behind it against the mechanism's own function."""
    cfg = copy.deepcopy(M.ODD)
    cfg["layers"] = [cfg["layers"][layer]]
    cfg.pop("loop")
    W = M.weights(cfg, 7)
    M.only(cfg, W, part)
    F, eps = M.f64(W), cfg["norm"]["eps"]
    ids = np.random.default_rng(8).integers(0, cfg["vocab"], 90)
    x, L = F["embed"][ids], cfg["layers"][0]
    norm = lambda v, name: K.layer_norm(v, F[name], F[name + ".b"], eps)
    if part == "mix":
        ref = x + norm(K.mixer(norm(x, "l0.norm1"), F, "l0.mix.", L, eps), "l0.norm1b")
    elif part == "mlp":
        ref = x + norm(K.gated_ffn(norm(x, "l0.norm2"), F, "l0.mlp."), "l0.norm2b")
    else:
        ref = x + K.token_side(x, F, "l0.", ids, 0, cfg["token_side"]["dim"], eps)
    m = R.Model.from_pretrained(folder(tmp_path, cfg, W), max_tokens=90, dtype=dtype, page_tokens=16)
    got = np.stack([m.decode_token_from_id(int(t)) for t in ids])
    assert np.abs(got - ref).max() / np.abs(ref).max() < (1e-5 if dtype == "f32" else 5e-3)
    logits = K.layer_norm(ref, F["final.norm"], F["final.norm.b"], eps) @ F["embed"].T
    m.set_len(0)
    assert M.error(all_logits(m, ids, [50, 40]), logits) < TOL[dtype]


def test_loop_vectors_alone(R, tmp_path):
    """Sublayers neutral: what is left is the embedding plus every pass's vector."""
    cfg = M.config(64, 90, [(M.lightning(2, 8, 8, (0.5, 0.9)), 16), (M.lightning(1, 8, 8, (0.5,)), None)], loop=(0, 1, 3), side=4)
    W = M.weights(cfg, 2)
    M.only(cfg, W, "none")
    ids = np.arange(30)
    ref = M.f64(W)["embed"][ids] + M.f64(W)["loop.step"].sum(axis=0)
    for dtype in ("f32", "bf16"):
        m = R.Model.from_pretrained(folder(tmp_path, cfg, W), max_tokens=30, dtype=dtype)
        got = np.stack([m.decode_token_from_id(int(t)) for t in ids])
        assert np.abs(got - ref).max() < 1e-5


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("window", [2, 11, 16, 63, 64, 65, 100])
def test_a_key_at_the_windows_edge(R, tmp_path, window, dtype):
    """A query that asks for the key at the far edge of its window, or one position beyond: in prompts, in portions and in
    decoding, at and away from page borders."""
    cfg, W, ids, places = M.edge_case(window)
    ref = K.forward(cfg, M.f64(W), ids)
    m = R.Model.from_pretrained(folder(tmp_path, cfg, W), max_tokens=len(ids), dtype=dtype, page_tokens=16)
    for portion in (None, 1, 77):
        m.set_len(0)
        got = all_logits(m, ids, portion)
        for kind in ("in", "out"):
            for p in places[kind]:
                assert M.error(got[p], ref[p]) < 3 * TOL[dtype], (kind, p, portion)
        assert M.error(got, ref) < 3 * TOL[dtype]


@pytest.mark.parametrize("kind", ["latent", "differential"])
@pytest.mark.parametrize("at", [0, 15, 16, 63, 64])
def test_a_far_key_and_the_first_tokens(R, tmp_path, at, kind):
    """No window: one key hundreds of positions back, at a page or tile border, stands out among all of them; the first
    tokens of a sequence have next to nothing to see."""
    mixer = M.latent(4, 16, 8, 24, 32, None, 1.0) if kind == "latent" else M.diff(4, 2, 20, 24, 1.0, M.rot(8, 100.0, M.SCALED), 0.3)
    cfg = M.config(64, 90, [(mixer, None)])
    W = M.weights(cfg, 6)
    M.point_query_at(cfg, W, 1, 2, strength=18.0)
    ids = np.random.default_rng(3).integers(3, 90, 800)
    asks = [70, 100, 764, 799]
    ids[asks] = 1
    lost = ids.copy()
    ids[at] = 2
    F = M.f64(W)
    ref = K.forward(cfg, F, ids)
    gone = K.forward(cfg, F, lost)
    assert min(M.error(gone[p], ref[p]) for p in asks) > 0.1
    path = folder(tmp_path, cfg, W)
    for dtype in ("f32", "bf16"):
        m = R.Model.from_pretrained(path, max_tokens=800, dtype=dtype, page_tokens=16)
        for portion in (None, [790] + [1] * 10, [64, 2, 700, 34]):
            m.set_len(0)
            got = all_logits(m, ids, portion)
            assert M.error(got[:12], ref[:12]) < 3 * TOL[dtype]
            assert M.error(got[asks], ref[asks]) < 3 * TOL[dtype]
            assert M.error(got, ref) < 3 * TOL[dtype]


def test_far_positions_keep_their_angles(R, tmp_path):
    """A rotated-only latent attention deep into a sequence: neighbouring positions' angles must be told apart there."""
    cfg = M.config(64, 90, [(M.latent(2, 4, 16, 16, 16, 20, 1.5, 3.0), None)])
    W = M.weights(cfg, 11)
    W["l0.mix.uk"] = np.zeros_like(W["l0.mix.uk"])
    ids = np.random.default_rng(5).integers(0, 90, 3000)
    ref = K.forward(cfg, M.f64(W), ids)
    path = folder(tmp_path, cfg, W)
    for dtype, portion in (("f32", [2900] + [1] * 100), ("bf16", None), ("bf16", [2990] + [1] * 10)):
        m = R.Model.from_pretrained(path, max_tokens=3000, dtype=dtype, use_graph=True)
        assert M.error(all_logits(m, ids, portion)[-100:], ref[-100:]) < 3 * TOL[dtype]


def test_the_state_recalls_across_a_thousand_tokens(R, tmp_path):
    """A decay close to one and one key far larger than the others: what was stored at the start decides the read-out a
    thousand tokens later; chunk borders and decoding keep it."""
    cfg = M.config(64, 90, [(M.lightning(2, 16, 24, (0.9995, 1.0)), None)])
    W = M.weights(cfg, 9)
    M.plain_norms(W, ["l0.norm1"])
    W["embed"][:, 0] = M.bf16(W["embed"][:, 1:].mean(axis=1))     # an entry that only the token to remember has
    W["embed"][2, 0] = 20.0
    W["l0.mix.k"] = M.bf16(W["l0.mix.k"] * 0.1)
    W["l0.mix.k"][:, 0] = M.bf16(np.linspace(20, 60, 32))
    ids = np.random.default_rng(4).integers(3, 90, 1000)
    ids[7] = 2
    F = M.f64(W)
    ref = K.forward(cfg, F, ids)
    lost = ids.copy()
    lost[7] = 3
    assert M.error(K.forward(cfg, F, lost)[-50:], ref[-50:]) > 0.2
    path = folder(tmp_path, cfg, W)
    for dtype, portion in (("f32", None), ("bf16", None), ("bf16", [2, 62, 65, 3, 700] + [1] * 168), ("f32", [500, 500])):
        m = R.Model.from_pretrained(path, max_tokens=1000, dtype=dtype)
        assert M.error(all_logits(m, ids, portion), ref) < 3 * TOL[dtype]


def test_wide_rows(R, tmp_path):
    """A width beyond one register pass of the norms' prologue, and a latent row too wide for the tensor-core attention."""
    for cfg, n in ((M.config(4608, 64, [(M.lightning(2, 16, 24, (0.5, 0.9)), 48), (M.diff(2, 1, 16, 16, 0.2, M.rot(8)), 16)], side=8), 20),
                   (M.config(64, 64, [(M.latent(3, 16, 8, 16, 1400, 9, 0.2), None)]), 40)):
        W = M.weights(cfg, 3)
        ids = np.random.default_rng(5).integers(0, cfg["vocab"], n)
        ref = K.forward(cfg, M.f64(W), ids)
        path = folder(tmp_path, cfg, W)
        for dtype in ("f32", "bf16"):
            m = R.Model.from_pretrained(path, max_tokens=64, dtype=dtype)
            one = np.stack([m.decode_token_logits_from_id(int(t)) for t in ids])
            assert M.error(one, ref) < 2 * TOL[dtype]
            m.set_len(0)
            assert M.error(all_logits(m, ids), ref) < 2 * TOL[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("width,side", [(64, 1), (200, 9), (1024, 300), (1024, 700)])
def test_token_side_sizes(R, tmp_path, width, side, dtype):
    """From one column per layer to widths of several GEMM tiles, at and off multiples of 8."""
    cfg = M.config(width, 90, [(M.lightning(2, 8, 12, (0.5, 0.9)), None), (M.latent(2, 8, 4, 8, 16, 9, 0.3), 24)], side=side)
    W = M.weights(cfg, 4)
    ids = np.random.default_rng(6).integers(0, 90, 40)
    ref = K.forward(cfg, M.f64(W), ids)
    assert M.error(K.forward(cfg, M.f64(W), ids, fault="first_part"), ref) > 0.1
    m = R.Model.from_pretrained(folder(tmp_path, cfg, W), max_tokens=40, dtype=dtype, use_graph=True)
    one = np.stack([m.decode_token_logits_from_id(int(t)) for t in ids])
    assert M.error(one, ref) < TOL[dtype]
    m.set_len(0)
    assert M.error(all_logits(m, ids, [30, 10]), ref) < TOL[dtype]


# ---------------------------------------------------------------------- sequences one after the other, rewinding
def test_cache_and_state_are_clean_for_the_next_sequence(R, made):
    cfg, _, path, ids, ref = made("ODD")
    other = np.random.default_rng(77).integers(0, cfg["vocab"], 150)
    used = R.Model.from_pretrained(path, max_tokens=200, page_tokens=16, use_graph=True)
    all_logits(used, other, [100, 1, 1, 48])
    used.set_len(0)
    a = all_logits(used, ids[:120], [90] + [1] * 30)
    fresh = R.Model.from_pretrained(path, max_tokens=200, page_tokens=16, use_graph=True)
    b = all_logits(fresh, ids[:120], [90] + [1] * 30)
    assert np.array_equal(a, b)
    assert M.error(a, ref[:120]) < TOL["bf16"]


def test_rewinding_goes_back_to_the_ends_of_prompt_passes(R, made):
    cfg, _, path, ids, ref = made("WIDE")
    m = R.Model.from_pretrained(path, max_tokens=200)
    m.prefill(ids[:60])
    m.prefill(ids[60:90])
    assert m.can_rewind(90) and m.can_rewind(60) and m.can_rewind(0) and not m.can_rewind(75)
    greedy = m.decode_steps_greedy(5, 20)
    with pytest.raises(R.CudaDecodeError, match="not kept"):
        m.set_len(100)
    m.set_len(90)
    assert np.array_equal(m.decode_steps_greedy(5, 20), greedy)
    m.set_len(60)
    got = all_logits(m, ids[60:130], [50, 1, 19])
    assert M.error(got, ref[60:130]) < TOL["bf16"]


def test_session_generates_what_the_oracle_generates(R, made):
    cfg, W, path, ids, _ = made("ODD")
    prompt = [int(t) for t in ids[:30]]
    want, gap = K.greedy(cfg, M.f64(W), prompt, 14)
    assert gap > 2e-2, "choose another prompt: a near tie"
    for dtype, graph in (("f32", False), ("bf16", True)):
        m = R.Model.from_pretrained(path, max_tokens=120, dtype=dtype, use_graph=graph)
        sess = R.InferenceSession(m, prompt)
        req = R.GenerationRequest("cuda", 14, 0.0, 1, 1, 1)
        assert sess.generate(req).results[0].sampled == want
        assert sess.generate(R.GenerationRequest("naive", 4, 0.0, 1, 1, 1)).results[0].sampled == want[:4]
        assert sess.generate(req).results[0].sampled == want            # after the naive request rewrote the cache
        half = R.InferenceSession(m, prompt[:18])
        assert half.generate_with_suffix(req, prompt[18:]).results[0].sampled == want


def test_sampled_requests_are_reproducible(R, made):
    cfg, _, path, ids, _ = made("WIDE")
    m = R.Model.from_pretrained(path, max_tokens=120, use_graph=True, max_samples=3)
    sess = R.InferenceSession(m, [int(t) for t in ids[:40]])
    for k in (8, 0, 40):
        many = sess.generate(R.GenerationRequest("cuda", 12, 9.0, k, 3, 5))
        alone = [sess.generate(R.GenerationRequest("cuda", 12, 9.0, k, 1, 5 + i)).results[0].sampled for i in range(3)]
        assert [r.sampled for r in many.results] == alone
        assert len({tuple(a) for a in alone}) > 1


def test_long_decoding_stays_on_the_oracle(R, made):
    cfg, W, path, _, _ = made("TAIL")
    ids = np.random.default_rng(12).integers(0, cfg["vocab"], 900)
    ref = K.forward(cfg, M.f64(W), ids)
    for dtype in ("f32", "bf16"):
        m = R.Model.from_pretrained(path, max_tokens=900, dtype=dtype, use_graph=True)
        got = all_logits(m, ids, [40] + [1] * 860)
        assert M.error(got[-100:], ref[-100:]) < TOL[dtype]


# ---------------------------------------------------------------------- loading, commands, errors
def test_loader_and_calls_report_what_is_wrong(R, tmp_path):
    cfg = M.ODD
    W = M.weights(cfg, 1)
    for name, change, message in (("l1.mix.dkv.norm", None, "missing tensor l1.mix.dkv.norm"), ("l0.norm1b.b", None, "missing tensor l0.norm1b.b"),
                                  ("loop.step", W["loop.step"][:-1], "shape"), ("side.embed", W["side.embed"][:, :-1], "shape"), ("l3.mix.uk", W["l3.mix.uk"][:-1], "shape")):
        bad = dict(W)
        if change is None:
            bad.pop(name)
        else:
            bad[name] = change
        with pytest.raises(R.CudaDecodeError, match=message):
            R.Model.from_pretrained(folder(tmp_path, cfg, bad))
    m = R.Model.from_pretrained(folder(tmp_path, cfg, W), max_tokens=16)
    with pytest.raises(R.CudaDecodeError, match="read the token id"):       # a hidden state does not say which token it is
        m.decode_token(np.zeros(cfg["width"], np.float32))
    with pytest.raises(R.CudaDecodeError, match="read the token id"):
        m.decode_token_argmax(np.zeros(cfg["width"], np.float32))
    assert m.len() == 0


def test_synthetic_configured_model_runs(R):
    m = R.Model.from_config(M.WIDE, 3, max_tokens=64)
    again = R.Model.from_config(M.WIDE, 3, max_tokens=64)
    a, b = m.prefill(list(range(40))), again.prefill(list(range(40)))
    assert np.isfinite(a).all() and np.array_equal(a, b) and a.std() > 0


def test_generate_command_takes_a_model_folder(R, made):
    cfg, W, path, ids, _ = made("ODD")
    prompt = [int(t) for t in ids[:30]]
    want, _ = K.greedy(cfg, M.f64(W), prompt, 8)
    out = subprocess.run([os.path.join(ROOT, "rustane_b200", "generate"), "--model", path, "--max-tokens", "64", "--prompt-ids", ",".join(map(str, prompt)),
                          "--decode-backend", "cuda", "--steps", "8", "--temperature", "0"], capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr[-2000:]
    line = [l for l in out.stdout.splitlines() if l.startswith("generated_ids=")][0]
    assert [int(t) for t in line.split("=")[1].split(",")] == want


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_runner_writes_what_the_model_computes(R, made, tmp_path, dtype):
    cfg, W, path, ids, ref = made("ODD")
    other = [int(t) for t in ids[::-1][:25]]
    ids = [int(t) for t in ids]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:70], "want": [0, 69, 33]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[70:73], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ids[73:74], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": other, "want": [24]}], "end": ["b"]}]
    out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "100"],
                         input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
    assert out.returncode == 0, out.stderr[-2000:]
    read = lambda k: np.fromfile(str(tmp_path / ("%d.f32" % k)), np.float32).reshape(-1, cfg["vocab"])
    tol = TOL["f32" if dtype == "float32" else "bf16"]
    assert M.error(read(0), ref[[0, 69, 33]]) < tol and M.error(read(2), ref[73:74]) < tol
    assert M.error(read(3), K.forward(cfg, M.f64(W), other)[24:]) < tol
