"""Small Kazodra configurations, random weights that let a fault show, and model folders for the tests."""
import numpy as np

from dafidra_models import bf16, error, f64, write_folder  # noqa: F401  (the folder format and the error measure are shared)
from oracle import kazodra_ref as K


def rot(dims, base=10000.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def latent(heads, dim, rot_dim, vdim, rank, window, scale, base=10000.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": rot(rot_dim, base)}
    if window:
        m["mask"] = {"size": window}
    return "latent_attention", m


def lightning(heads, dim, vdim, decay):
    return "lightning", {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def diff(heads, kv_heads, dim, vdim, scale, rotation, d=0.4):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rotation, "diff": d}


def config(width, vocab, layers, loop=None, side=None, eps=3e-5):
    c = {"architecture": "Kazodra", "width": width, "vocab": vocab, "norm": {"eps": eps},
         "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (t, m), ff in layers]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    if side:
        c["token_side"] = {"dim": side}
    return c


def shapes(cfg):
    D, out = cfg["width"], {}

    def norm(name):
        out[name], out[name + ".b"] = (D,), (D,)

    out["embed"] = (cfg["vocab"], D)
    side = (cfg.get("token_side") or {}).get("dim", 0)
    if side:
        out["side.embed"] = (cfg["vocab"], side * len(cfg["layers"]))
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], D)
    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, c = "l%d." % i, L["mixer"]
        m, H, vd = p + "mix.", c["heads"], c["vdim"]
        norm(p + "norm1"), norm(p + "norm1b")
        out[m + "o"] = (D, H * vd)
        if L["type"] == "latent_attention":
            out.update({m + "q": (H * (c["dim"] + c["rot_dim"]), D), m + "dkv": (c["kv_rank"] + c["rot_dim"], D), m + "dkv.norm": (c["kv_rank"],),
                        m + "uk": (H * c["dim"], c["kv_rank"]), m + "uv": (H * vd, c["kv_rank"])})
        elif L["type"] == "lightning":
            out.update({m + "q": (H * c["dim"], D), m + "k": (H * c["dim"], D), m + "v": (H * vd, D), m + "g": (H * vd, D), m + "norm": (H * vd,)})
        else:
            G = c["kv_heads"]
            out.update({m + "q": (H * 2 * c["dim"], D), m + "k": (G * 2 * c["dim"], D), m + "v": (G * vd, D), m + "g": (H * vd, D)})
            out.update({m + n: (c["dim"],) for n in ("lq1", "lk1", "lq2", "lk2")})
        if L["mlp"]:
            norm(p + "norm2"), norm(p + "norm2b")
            out.update({p + "mlp.gate": (L["mlp"]["ff"], D), p + "mlp.up": (L["mlp"]["ff"], D), p + "mlp.down": (D, L["mlp"]["ff"])})
        if side:
            out.update({p + "side.gate": (side, D), p + "side.proj": (D, side), p + "side.norm": (D,)})
    return out


def weights(cfg, seed):
    """bf16-representable random weights: unit-variance projections, norm weights and biases away from their neutral value,
    an embedding and loop vectors whose mean is not zero, a second map whose weight is well away from `diff`."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in shapes(cfg).items():
        x = rng.standard_normal(shape)
        leaf = name.split(".")[-1]
        if name in ("embed", "loop.step"):
            x = x + 0.5
        elif name == "side.embed":
            pass
        elif leaf == "b":
            x = 0.3 * x
        elif leaf.startswith("norm"):
            x = 1.0 + 0.3 * x
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            x = 0.8 * x / np.sqrt(np.sqrt(shape[0]))
        else:
            x = x / np.sqrt(shape[1])
        W[name] = bf16(x)
    return W


def only(cfg, W, part):
    """Neutralise the other sublayers of every layer: `part` is mix, mlp or side."""
    for name in W:
        p = name.split(".")
        which = {"norm1b": "mix", "norm2b": "mlp"}.get(p[1] if len(p) > 1 else "", "side" if name.endswith("side.norm") else None)
        if which and which != part:
            W[name] = np.zeros_like(W[name])


def plain_norms(W, names):
    for n in names:
        W[n], W[n + ".b"] = np.ones_like(W[n]), np.zeros_like(W[n])


def point_query_at(cfg, W, asker, needle, strength):
    """Change layer 0's query projection so that token `asker`'s query is, in the entries that are not rotated, token
    `needle`'s key in every head (and map) and zero in the others: one score stands out at any distance, so a key lost or
    gained shows in the logits."""
    L, p = cfg["layers"][0], "l0.mix."
    c = L["mixer"]
    plain_norms(W, ["l0.norm1"])
    F = f64(W)
    h = K.layer_norm(F["embed"], F["l0.norm1"], F["l0.norm1.b"], cfg["norm"]["eps"])
    if L["type"] == "latent_attention":
        lat = K.rms((F[p + "dkv"] @ h[needle])[:c["kv_rank"]], cfg["norm"]["eps"]) * F[p + "dkv.norm"]
        key = (F[p + "uk"] @ lat).reshape(c["heads"], c["dim"])
        want = np.concatenate([key, np.zeros((c["heads"], c["rot_dim"]))], axis=1)
    else:
        key = (F[p + "k"] @ h[needle]).reshape(c["kv_heads"], 2, c["dim"]).copy()
        key[..., :c["rot"]["dims"]] = 0.0
        want = np.repeat(key, c["heads"] // c["kv_heads"], axis=0)
    # of one length, so that every head's score stands out the same
    n = np.sqrt((want ** 2).sum(axis=-1, keepdims=True))
    want = (want / n ** 2 * strength).reshape(-1)
    u = h[asker] / np.dot(h[asker], h[asker])
    W[p + "q"] = bf16(W[p + "q"] + np.outer(want - F[p + "q"] @ h[asker], u))


def edge_case(window, seed=4):
    """One latent layer with a window and nothing else, and a sequence in which a token asks for one that stands exactly at
    the window's far edge ("in") or one position beyond it ("out"), at and away from page borders."""
    cfg = config(64, 90, [(latent(4, 16, 8, 24, 32, window, 1.0), None)])
    W = weights(cfg, seed)
    point_query_at(cfg, W, asker=1, needle=2, strength=12.0)
    step = window + 9
    ids = np.random.default_rng(seed).integers(3, cfg["vocab"], 16 * step)
    places = {"in": [], "out": []}
    for n in range(7):
        p = 2 * n * step + step + 3
        for kind, d, at in (("in", window - 1, p), ("out", window, p + step)):
            ids[at], ids[at - d] = 1, 2
            places[kind].append(at)
    return cfg, W, ids, places


SCALED = (4.0, 1.0, 3.0, 40)
ODD = config(96, 301, [                                   # sizes that share no factor, every kind of layer, three passes
    (diff(6, 2, 12, 20, 0.31, rot(8, 500.0, SCALED)), 72),
    (latent(5, 20, 12, 28, 40, 13, 0.2, 300.0), None),
    (lightning(3, 20, 36, (0.0, 0.71, 1.0)), 44),
    (latent(18, 8, 4, 12, 24, None, 0.35), 30),
    (lightning(2, 70, 75, (0.93, 0.4)), None),
], loop=(1, 4, 3), side=10)
WIDE = config(256, 520, [                                 # head widths of real models; the whole stack runs twice
    (latent(4, 64, 32, 64, 512, 90, 0.1), 320),
    (diff(4, 2, 64, 128, 0.125, rot(64, 50000.0, (8.0, 1.0, 4.0, 64)), 0.7), 256),
    (lightning(2, 128, 128, (0.97, 0.995)), 128),
], loop=(0, 3, 2), side=32, eps=1e-5)
BROAD = config(128, 200, [(latent(2, 192, 64, 256, 528, 40, 0.06), 128), (diff(2, 1, 144, 200, 0.08, rot(144)), None), (lightning(1, 200, 264, (0.9,)), 64)], eps=1e-5)
PLAIN = config(64, 130, [                                 # no loop, no token side, one head of everything
    (lightning(1, 16, 8, (0.8,)), None),
    (diff(1, 1, 16, 16, 0.3, rot(16), 0.2), None),
    (latent(1, 16, 2, 8, 16, 1, 0.3), 16),
])
TAIL = config(72, 57, [                                   # the loop ends ahead of the last layer and runs once; narrow side
    (latent(3, 12, 6, 20, 136, 30, 0.3), 20),
    (diff(3, 3, 20, 28, 0.25, rot(4, 100.0)), 24),
    (lightning(5, 6, 10, (0.99, 0.9, 0.5, 0.999, 0.1)), None),
], loop=(1, 2, 1), side=1, eps=1e-4)
RAGGED = config(91, 75, [                                 # a width that fits no chunk
    (diff(2, 1, 10, 14, 0.3, rot(6, 200.0)), 17),
    (latent(3, 9, 2, 11, 21, 7, 0.3), None),
    (lightning(3, 7, 5, (0.9, 0.6, 0.97)), 23),
], loop=(0, 2, 2), side=3)
