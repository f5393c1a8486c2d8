"""The Dafidra decoder on the GPU against its plain restatement (oracle/dafidra_ref.py): each mechanism alone, whole models,
prompt passes against token-by-token decoding, portions, rewinding, generation, and the trace runner."""
import copy
import json
import os
import subprocess

import numpy as np
import pytest

import dafidra_models as M
from oracle import dafidra_ref as D

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# fp32: summation order only.  bf16 weights (exact in both): fp16 cache rows and 16 + 16 bit GEMM operands; KEPT is the
# distance to an oracle whose cache rounds its rows the same way, where only the operands' rounding is left.
TOL = {"f32": 2e-5, "bf16": 1e-2}
KEPT = 2e-3
SEED = {"ODD": 2, "WIDE": 5, "BROAD": 1, "LAST_MIXER": 1, "NARROW": 37, "RAGGED": 2}   # routing margins above 1e-2 on the sequences used here


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
            margins = []
            ref = D.forward(cfg, M.f64(W), ids, margins=margins)
            assert not margins or min(margins) > 1e-2, "choose another seed: a routing choice is a close call"
            cache[name] = cfg, W, path, ids, ref
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
@pytest.mark.parametrize("name", ["ODD", "WIDE", "BROAD", "LAST_MIXER", "NARROW", "RAGGED"])
def test_whole_prompt_and_decoding_match_the_oracle(R, made, name, dtype):
    cfg, _, path, ids, ref = made(name)
    m = R.Model.from_pretrained(path, max_tokens=256, dtype=dtype, page_tokens=16)
    got = all_logits(m, ids)
    assert M.error(got, ref) < TOL[dtype], M.error(got, ref)
    assert m.len() == len(ids)
    m.set_len(0)
    one = np.stack([m.decode_token_logits_from_id(int(t)) for t in ids])
    assert M.error(one, ref) < TOL[dtype], M.error(one, ref)
    if dtype == "bf16":
        rounded = D.forward(cfg, M.f64(made(name)[1]), ids, cache=np.float16)
        print(name, "to the oracle:", M.error(got, ref), M.error(one, ref), "with rounded cache rows:", M.error(got, rounded), M.error(one, rounded))
        assert M.error(got, rounded) < KEPT and M.error(one, rounded) < KEPT


@pytest.mark.parametrize("name,portions", [
    ("ODD", [2] * 100), ("ODD", [9, 2, 13, 8, 64, 3, 65, 2, 34]), ("WIDE", [63, 2, 64, 1, 65, 5]), ("LAST_MIXER", [8] * 25), ("BROAD", [130, 3, 50, 2, 15]), ("NARROW", [2, 11, 100, 1, 86]), ("RAGGED", [50, 2, 9, 1, 138]),
])
def test_portions_of_a_prompt_do_not_change_its_logits(R, made, name, portions):
    cfg, _, path, ids, ref = made(name)
    m = R.Model.from_pretrained(path, max_tokens=200, page_tokens=32, use_graph=True)
    assert M.error(all_logits(m, ids, list(portions)), ref) < TOL["bf16"]


def test_long_prompts_are_processed_in_pieces(R, made, monkeypatch):
    cfg, _, path, ids, ref = made("ODD")
    monkeypatch.setenv("CD_PREFILL_ROWS", "70")
    m = R.Model.from_pretrained(path, max_tokens=200)
    assert M.error(all_logits(m, ids), ref) < TOL["bf16"]


def test_bf16_cache_and_single_rounding_options(R, made, monkeypatch):
    cfg, _, path, ids, ref = made("WIDE")
    m = R.Model.from_pretrained(path, max_tokens=200, kv_dtype="bf16")
    assert M.error(all_logits(m, ids, [150, 2, 48]), ref) < 2e-2
    monkeypatch.setenv("CD_PREFILL", "fast")
    m.set_len(0)
    assert M.error(all_logits(m, ids), ref) < 5e-2


# ---------------------------------------------------------------------- each mechanism alone
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("part", ["left", "right", "mlp"])
@pytest.mark.parametrize("layer", [0, 1])
def test_each_mechanism_alone(R, tmp_path, layer, part, dtype):
    """One layer of ODD with the others neutral: the hidden state behind it against the mechanism's own function."""
    cfg = copy.deepcopy(M.ODD)
    cfg["layers"] = [cfg["layers"][layer]]
    if part != "mlp":
        cfg["layers"][0]["mlp"] = None
    W = M.weights(cfg, 7)
    M.only(cfg, W, part)
    F, eps, mult = M.f64(W), cfg["norm"]["eps"], cfg["residual_mult"]
    ids = np.random.default_rng(8).integers(0, cfg["vocab"], 90)
    x = F["embed"][ids]
    L = cfg["layers"][0]
    if part == "left":
        y = 0.5 * D.norm_plain(D.attention(x, F, "l0.mix.left.", L["mixer"]["left"], eps), F["l0.mix.left.out"], eps)
    elif part == "right":
        y = 0.5 * D.norm_plain(D.matrix_memory(x, F, "l0.mix.right.", L["mixer"]["right"], eps), F["l0.mix.right.out"], eps)
    else:
        y = D.feed_forward(x, F, "l0.mlp.", L["mlp"])
    ref = x + mult * D.norm_around_zero(y, F["l0.norm1" if part != "mlp" else "l0.norm2"], eps)
    m = R.Model.from_pretrained(folder(tmp_path, cfg, W), max_tokens=90, dtype=dtype, page_tokens=16)
    got = np.stack([m.decode_token_from_id(int(t)) for t in ids])
    assert np.abs(got - ref).max() / np.abs(ref).max() < (1e-5 if dtype == "f32" else 3e-3)
    logits = D.norm_around_zero(ref, F["final.norm"], eps) @ F["head"].T
    m.set_len(0)
    assert M.error(all_logits(m, ids, [50, 40]), logits) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("window", [1, 2, 11, 32, 64, 65, 100])
def test_a_key_at_the_windows_edge(R, tmp_path, window, dtype):
    """A query that asks for the key at the far edge of its window, or one position beyond: in prompts, in portions and in
    decoding, at and away from page borders."""
    cfg, W, ids, places = M.window_case(max(window, 2)) if window > 1 else M.window_case(2)
    if window == 1:
        cfg["layers"][0]["mixer"]["left"]["mask"]["size"] = 1
    ref = D.forward(cfg, M.f64(W), ids)
    m = R.Model.from_pretrained(folder(tmp_path, cfg, W), max_tokens=len(ids), dtype=dtype, page_tokens=16)
    for portion in (None, 1, 77):
        m.set_len(0)
        got = all_logits(m, ids, portion)
        for kind in ("in", "out"):
            for p in places[kind]:
                assert M.error(got[p], ref[p]) < 3 * TOL[dtype], (kind, p, portion)
        assert M.error(got, ref) < 3 * TOL[dtype]


def test_a_far_key_without_a_window_and_the_first_tokens(R, tmp_path):
    """No window: a key 700 positions back, at a page border, stands out among all of them; the first tokens of a sequence
    see hardly anything but the sink."""
    cfg = M.config(64, 90, [(M.attn(4, 2, 16, 24, None, 3.0, 0.05, 100), M.memory(2, 8, 8, 6.0), None)])
    W = M.weights(cfg, 6)
    M.only(cfg, W, "left")
    M.point_query_at(cfg, W, 0, 1, 2, strength=4.0)
    ids = np.random.default_rng(3).integers(3, 90, 800)
    for at in (0, 15, 16, 63, 64):
        ids[at] = 2
    asks = [5, 100, 764, 799]
    ids[asks] = 1
    F = M.f64(W)
    ref = D.forward(cfg, F, ids)
    lost = ids.copy()
    lost[[0, 15, 16, 63, 64]] = 3
    assert M.error(D.forward(cfg, F, lost)[asks[1:]], ref[asks[1:]]) > 0.05   # the far keys show
    path = folder(tmp_path, cfg, W)
    for dtype in ("f32", "bf16"):
        m = R.Model.from_pretrained(path, max_tokens=800, dtype=dtype, page_tokens=16)
        for portion in (None, [790] + [1] * 10):
            m.set_len(0)
            got = all_logits(m, ids, portion)
            assert M.error(got[:12], ref[:12]) < 3 * TOL[dtype]
            assert M.error(got[asks], ref[asks]) < 3 * TOL[dtype]
            assert M.error(got, ref) < 3 * TOL[dtype]


def test_the_memory_recalls_across_a_thousand_tokens(R, tmp_path):
    """Forget gates almost fully open and one input gate far above the others: what was stored at the start decides the
    read-out a thousand tokens later; chunk borders and decoding keep it."""
    cfg = M.config(64, 90, [(M.attn(2, 1, 16, 16, 8, 0.3), M.memory(2, 16, 24, 12.0), None)])
    W = M.weights(cfg, 9)
    M.only(cfg, W, "right")
    p = "l0.mix.right."
    W[p + "f.b"][:] = 9.0
    W[p + "i.b"][:] = -3.0
    u = W["embed"][2] / np.dot(W["embed"][2], W["embed"][2])
    W[p + "i"] = M.bf16(W[p + "i"] * 0.1 + 9.0 * u)
    ids = np.random.default_rng(4).integers(3, 90, 1000)
    ids[7] = 2
    F = M.f64(W)
    ref = D.forward(cfg, F, ids)
    lost = ids.copy()
    lost[7] = 3
    assert M.error(D.forward(cfg, F, lost)[-50:], ref[-50:]) > 0.3
    path = folder(tmp_path, cfg, W)
    for dtype, portion in (("f32", None), ("bf16", None), ("bf16", [2, 62, 65, 3, 700] + [1] * 168), ("f32", [500, 500])):
        m = R.Model.from_pretrained(path, max_tokens=1000, dtype=dtype)
        assert M.error(all_logits(m, ids, portion), ref) < 3 * TOL[dtype]


def test_wide_rows_take_the_plain_expert_kernels(R, tmp_path):
    """More expert columns per token than the streamed GEMV keeps in registers, and a width beyond one register pass."""
    for cfg, n in ((M.config(64, 80, [(M.attn(2, 1, 16, 16, 8, 0.3), M.memory(2, 16, 24, 12.0), M.moe(9, 9, 1100, (3, 3)))]), 12),
                   (M.config(4608, 64, [(M.attn(2, 1, 16, 16, 8, 0.3), M.memory(2, 16, 24, 12.0), M.dense(48))]), 20)):
        W = M.weights(cfg, 3)
        ids = np.random.default_rng(5).integers(0, cfg["vocab"], n)
        ref = D.forward(cfg, M.f64(W), ids)
        path = folder(tmp_path, cfg, W)
        for dtype in ("f32", "bf16"):
            m = R.Model.from_pretrained(path, max_tokens=32, dtype=dtype)
            one = np.stack([m.decode_token_logits_from_id(int(t)) for t in ids])
            assert M.error(one, ref) < 2 * TOL[dtype]
            m.set_len(0)
            assert M.error(all_logits(m, ids), ref) < 2 * TOL[dtype]


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
    assert not m.can_rewind(100)
    with pytest.raises(R.CudaDecodeError, match="not kept"):
        m.set_len(100)
    m.set_len(90)
    assert np.array_equal(m.decode_steps_greedy(5, 20), greedy)
    m.set_len(60)
    assert not m.can_rewind(90)                     # what follows may be another continuation
    got = all_logits(m, ids[60:130], [50, 1, 19])
    assert M.error(got, ref[60:130]) < TOL["bf16"]
    for k in range(6):                              # more ends than are kept: the latest ones stay
        m.prefill(ids[130 + 10 * k:140 + 10 * k])
    assert m.can_rewind(190) and m.can_rewind(180) and not m.can_rewind(130)


def test_session_generates_what_the_oracle_generates(R, made):
    cfg, W, path, ids, _ = made("ODD")
    prompt = [int(t) for t in ids[:30]]
    want, gap = D.greedy(cfg, M.f64(W), prompt, 14)
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
        seen = []
        half.generate_stream_with_suffix(req, prompt[18:], lambda tok, s, g: seen.append(tok))
        assert seen == want


def test_sampled_requests_are_reproducible_and_independent_of_each_other(R, made):
    """Several samples of one request, one after the other from the shared prompt: each equals the request for it alone."""
    cfg, _, path, ids, _ = made("WIDE")
    m = R.Model.from_pretrained(path, max_tokens=120, use_graph=True, max_samples=3)
    sess = R.InferenceSession(m, [int(t) for t in ids[:40]])
    for k in (8, 0, 40):
        many = sess.generate(R.GenerationRequest("cuda", 12, 0.9, k, 3, 5))
        assert many.decode_selection.mode == "kv_cache_cuda"
        alone = [sess.generate(R.GenerationRequest("cuda", 12, 0.9, k, 1, 5 + i)).results[0].sampled for i in range(3)]
        assert [r.sampled for r in many.results] == alone
        assert len({tuple(a) for a in alone}) > 1
    with pytest.raises(R.CudaDecodeError):
        m.decode_steps_samples([1, 2], 4)


def test_long_decoding_stays_on_the_oracle(R, made):
    cfg, W, path, _, _ = made("LAST_MIXER")
    ids = np.random.default_rng(12).integers(0, cfg["vocab"], 900)
    ref = D.forward(cfg, M.f64(W), ids)
    for dtype in ("f32", "bf16"):
        m = R.Model.from_pretrained(path, max_tokens=900, dtype=dtype, use_graph=True)
        got = all_logits(m, ids, [40] + [1] * 860)
        assert M.error(got[-100:], ref[-100:]) < TOL[dtype]


# ---------------------------------------------------------------------- loading, commands, errors
def test_loader_reports_missing_and_misshapen_tensors(R, tmp_path):
    cfg = M.LAST_MIXER
    W = M.weights(cfg, 1)
    for name, change, message in (("l1.mix.right.i.b", None, "missing tensor l1.mix.right.i.b"), ("l0.mix.left.o", W["l0.mix.left.o"][:-1], "shape"),
                                  ("embed", W["embed"][:, :-2], "shape")):
        bad = dict(W)
        if change is None:
            bad.pop(name)
        else:
            bad[name] = change
        with pytest.raises(R.CudaDecodeError, match=message):
            R.Model.from_pretrained(folder(tmp_path, cfg, bad))
    path = folder(tmp_path, cfg, W)
    with open(os.path.join(path, "model.safetensors"), "r+b") as f:
        f.truncate(os.path.getsize(f.name) - 10)
    with pytest.raises(R.CudaDecodeError, match="outside the file"):
        R.Model.from_pretrained(path)
    with pytest.raises(R.CudaDecodeError, match="f32 or bf16"):
        R.Model.from_pretrained(folder(tmp_path, cfg, W), dtype="fp8")
    m = R.Model.from_pretrained(folder(tmp_path, cfg, W), max_tokens=16)
    with pytest.raises(R.CudaDecodeError, match="cfg.seq"):
        m.prefill(list(range(17)))
    with pytest.raises(R.CudaDecodeError, match="vocab"):
        m.prefill([cfg["vocab"]])
    with pytest.raises(R.CudaDecodeError, match="behind the last token"):
        m.prefill_logits([1, 2, 3], [3])
    assert m.len() == 0


def test_synthetic_configured_model_runs(R):
    m = R.Model.from_config(M.WIDE, 3, max_tokens=64)
    again = R.Model.from_config(M.WIDE, 3, max_tokens=64)
    a, b = m.prefill(list(range(40))), again.prefill(list(range(40)))
    assert np.isfinite(a).all() and np.array_equal(a, b) and a.std() > 0


def test_generate_command_takes_a_model_folder(R, made):
    cfg, W, path, ids, _ = made("ODD")
    prompt = [int(t) for t in ids[:30]]
    want, _ = D.greedy(cfg, M.f64(W), prompt, 8)
    out = subprocess.run([os.path.join(ROOT, "rustane_b200", "generate"), "--model", path, "--max-tokens", "64", "--prompt-ids", ",".join(map(str, prompt)),
                          "--decode-backend", "cuda", "--steps", "8", "--temperature", "0"], capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr[-2000:]
    line = [l for l in out.stdout.splitlines() if l.startswith("generated_ids=")][0]
    assert [int(t) for t in line.split("=")[1].split(",")] == want


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_runner_writes_what_the_model_computes(R, made, tmp_path, dtype):
    cfg, _, path, ids, ref = made("LAST_MIXER")
    other = [int(t) for t in ids[::-1][:25]]
    ids = [int(t) for t in ids]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:70], "want": [0, 69, 33]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[70:73], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ids[73:74], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": other, "want": [24]}], "end": ["b"]}]
    out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "100"],
                         input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
    assert out.returncode == 0, out.stderr[-2000:]
    assert [l for l in out.stdout.splitlines() if l.startswith("done")] == ["done %d" % k for k in range(4)]
    read = lambda k: np.fromfile(str(tmp_path / ("%d.f32" % k)), np.float32).reshape(-1, cfg["vocab"])
    tol = TOL["f32" if dtype == "float32" else "bf16"]
    assert M.error(read(0), ref[[0, 69, 33]]) < tol and M.error(read(2), ref[73:74]) < tol
    assert not os.path.exists(str(tmp_path / "1.f32"))
    W = M.f64(M.weights(cfg, SEED["LAST_MIXER"]))
    assert M.error(read(3), D.forward(cfg, W, other)[24:]) < tol
