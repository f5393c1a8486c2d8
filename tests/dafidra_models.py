"""Small Dafidra configurations, random weights that let a fault show, and model folders for the tests."""
import json
import os

import numpy as np


def attn(heads, kv_heads, dim, vdim, window, scale, coef=0.4, every=7):
    a = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "q_temp": {"coef": coef, "every": every}}
    if window:
        a["mask"] = {"size": window}
    return a


def memory(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def config(width, vocab, layers, eps=3e-4, mult=0.7):
    return {"architecture": "Dafidra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": [{"type": "parallel", "mixer": {"left": a, "right": m}, "mlp": f} for a, m, f in layers]}


def bf16(x):
    """Round to bfloat16, kept as float32 values."""
    u = np.asarray(x, np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32)


def shapes(cfg):
    D, out = cfg["width"], {}
    out["embed"] = out["head"] = (cfg["vocab"], D)
    out["final.norm"] = (D,)
    for i, L in enumerate(cfg["layers"]):
        p, a, m, f = "l%d." % i, L["mixer"]["left"], L["mixer"]["right"], L["mlp"]
        q, k, v = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]
        out[p + "norm1"] = (D,)
        pl, pr = p + "mix.left.", p + "mix.right."
        out.update({pl + "q": (q, D), pl + "k": (k, D), pl + "v": (v, D), pl + "q.norm": (q,), pl + "k.norm": (k,), pl + "sink": (a["heads"],),
                    pl + "g": (a["heads"], D), pl + "o": (D, a["heads"] * a["vdim"]), pl + "out": (D,)})
        qk, mv, H = m["heads"] * m["dim"], m["heads"] * m["vdim"], m["heads"]
        out.update({pr + "q": (qk, D), pr + "k": (qk, D), pr + "v": (mv, D), pr + "g": (mv, D), pr + "o": (D, mv), pr + "norm": (mv,),
                    pr + "i": (H, D), pr + "i.b": (H,), pr + "f": (H, D), pr + "f.b": (H,), pr + "out": (D,)})
        if f is None:
            continue
        out[p + "norm2"] = (D,)
        ffn = lambda q: {q + "gate": (f_ff, D), q + "up": (f_ff, D), q + "down": (D, f_ff)}
        if f["kind"] == "dense":
            f_ff = f["ff"]
            out.update(ffn(p + "mlp."))
        else:
            f_ff = f["expert"]["ff"]
            out[p + "mlp.router"] = (f["router"]["experts"], D)
            for e in range(f["router"]["experts"]):
                out.update(ffn("%smlp.e%d." % (p, e)))
    return out


def weights(cfg, seed):
    """bf16-representable random weights: unit-variance projections, norm weights away from their neutral value, sinks that
    take a real share, forget gates mostly open, a router with clear preferences."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in shapes(cfg).items():
        x = rng.standard_normal(shape)
        leaf = name.split(".")[-1]
        if name == "embed":
            pass
        elif name == "head":
            x = x / np.sqrt(shape[1])
        elif leaf in ("norm1", "norm2") or name == "final.norm":
            x = 0.3 * x
        elif leaf == "norm" or leaf == "out":
            x = 1.0 + 0.3 * x
        elif leaf == "sink":
            x = 1.0 + x
        elif name.endswith("i.b"):
            x = 0.5 * x
        elif name.endswith("f.b"):
            x = 2.5 + x
        elif leaf == "router":
            x = (3.0 if shape[0] < 32 else 12.0) * x / np.sqrt(shape[1])
        else:
            x = x / np.sqrt(shape[1])
        W[name] = bf16(x)
    return W


def write_folder(path, cfg, W):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, at, blobs = {}, 0, []
    for name, x in W.items():
        b = (np.ascontiguousarray(bf16(x)).view(np.uint32) >> 16).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(x.shape), "data_offsets": [at, at + len(b)]}
        at += len(b)
        blobs.append(b)
    h = json.dumps(header).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(len(h).to_bytes(8, "little") + h + b"".join(blobs))
    return str(path)


def f64(W):
    return {k: v.astype(np.float64) for k, v in W.items()}


def error(got, ref):
    """Largest root-mean-square difference of a row, means taken off, over the root mean square of the reference."""
    got, ref = np.atleast_2d(np.asarray(got, np.float64)), np.atleast_2d(np.asarray(ref, np.float64))
    d = got - ref
    d = d - d.mean(axis=1, keepdims=True)
    r = ref - ref.mean(axis=1, keepdims=True)
    return float(np.sqrt((d * d).mean(axis=1)).max() / np.sqrt((r * r).mean()))


def point_query_at(cfg, W, layer, asker, needle, strength=1.0):
    """Change one layer's query projection so that token `asker`'s query is the key of token `needle` in every head (the
    layer's input being the embedding): one score stands out, so a key lost or gained shows in the logits."""
    a = cfg["layers"][layer]["mixer"]["left"]
    p = "l%d.mix.left." % layer
    E, K, Q = W["embed"], W[p + "k"], W[p + "q"]
    u = E[asker] / np.dot(E[asker], E[asker])
    key = (K @ E[needle]).reshape(a["kv_heads"], a["dim"])
    want = np.repeat(key, a["heads"] // a["kv_heads"], axis=0).reshape(-1) * strength
    W[p + "q"] = bf16(Q + np.outer(want - Q @ E[asker], u))
    W[p + "q.norm"] = np.ones_like(W[p + "q.norm"])
    W[p + "k.norm"] = np.ones_like(W[p + "k.norm"])


def only(cfg, W, part):
    """Neutralise the other mechanisms of every layer: `part` is left, right or mlp."""
    for i in range(len(cfg["layers"])):
        for side in ("left", "right"):
            if side != part:
                W["l%d.mix.%s.out" % (i, side)] = np.zeros_like(W["l%d.mix.%s.out" % (i, side)])


def window_case(window, seed=4):
    """One attention layer (the other mechanisms neutral), and a sequence in which a token asks for one that stands exactly
    at the window's far edge ("in") or one position beyond it ("out"), away from and at page borders."""
    cfg = config(64, 90, [(attn(4, 2, 16, 24, window, 2.0, 0.1, 40), memory(2, 8, 8, 6.0), None)])
    W = weights(cfg, seed)
    only(cfg, W, "left")
    point_query_at(cfg, W, 0, asker=1, needle=2)
    rng = np.random.default_rng(seed)
    step = window + 9
    ids = rng.integers(3, cfg["vocab"], 16 * step)
    places = {"in": [], "out": []}
    for n in range(8):
        p = 2 * n * step + step + 3
        for kind, d, at in (("in", window - 1, p), ("out", window, p + step)):
            if at < len(ids):
                ids[at], ids[at - d] = 1, 2
                places[kind].append(at)
    return cfg, W, ids, places


ODD = config(96, 301, [                                   # sizes that share no factor; every kind of layer
    (attn(6, 3, 24, 20, 13, 0.31), memory(3, 20, 36, 9.0), dense(72)),
    (attn(3, 1, 40, 44, 37, 0.2, 0.25, 16), memory(5, 12, 20, 6.0), moe(12, 3, 40, (4, 2))),
    (attn(2, 2, 16, 24, None, 0.4, 0.6, 5), memory(1, 28, 52, 12.0), None),
    (attn(5, 5, 8, 12, 1, 0.5, 0.1, 3), memory(2, 16, 8, 20.0), moe(6, 1, 24)),
])
WIDE = config(256, 520, [                                 # head widths of real models
    (attn(4, 2, 128, 64, 90, 0.09, 0.3, 32), memory(2, 128, 160, 15.0), moe(8, 4, 96, (2, 1))),
    (attn(2, 1, 64, 128, 64, 0.125, 0.2, 50), memory(2, 64, 96, 15.0), dense(320)),
], eps=1e-5, mult=0.4)
BROAD = config(128, 200, [(attn(2, 1, 192, 256, 48, 0.07), memory(1, 200, 264, 10.0), dense(128))], eps=1e-5, mult=1.0)
LAST_MIXER = config(64, 130, [(attn(4, 2, 16, 16, 20, 0.3), memory(2, 16, 32, 8.0), None), (attn(1, 1, 32, 48, 9, 0.2), memory(4, 8, 12, 8.0), None)], mult=0.9)
NARROW = config(72, 57, [                                 # widths that are no multiple of a GEMM chunk, many small experts
    (attn(3, 3, 12, 4, 6, 0.6, 0.2, 2), memory(3, 6, 10, 7.0), moe(40, 6, 12, (10, 7))),
    (attn(4, 1, 20, 28, 150, 0.25), memory(1, 4, 100, 7.0), dense(20)),
], eps=1e-4, mult=0.6)
RAGGED = config(61, 75, [                                 # a width that fits no chunk
    (attn(3, 1, 12, 10, 9, 0.5, 0.2, 4), memory(2, 9, 7, 7.0), moe(6, 2, 11)),
    (attn(2, 2, 20, 6, None, 0.25), memory(3, 5, 12, 9.0), dense(19)),
    (attn(1, 1, 8, 8, 5, 0.4), memory(1, 4, 4, 7.0), None),
], eps=1e-4, mult=0.8)
