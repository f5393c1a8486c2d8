"""A plain numpy restatement of the Kazodra decoder (TEST INFRASTRUCTURE ONLY).

One function per mechanism, written for one sequence at a time, token by token where the mechanism is a
recurrence and over the whole sequence where it is not.  Nothing here is shared with the product: no kernel,
no loader, no cache.  Weights are a dict name -> float array (matrices [out, in]); the configuration is the
dict a config.json holds.  All arithmetic is in the arrays' own type (float64 in the tests), so that a
comparison measures the product's rounding and not this file's.

`fault` names a deliberate mistake to make in one mechanism; tests use it to show that their inputs would
expose that mistake.  `cache` (a numpy type) rounds what a cache keeps to what one of that type holds.
"""
import numpy as np


def rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps, fault=""):
    m = 0.0 if fault == "norm_keeps_mean" else x.mean(axis=-1, keepdims=True)
    c = x - m
    y = c / np.sqrt(np.mean(c * c, axis=-1, keepdims=True) + eps) * w
    return y if fault == "norm_no_bias" else y + b


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot, fault=""):
    """One angular frequency per pair; `scaling` stretches the wavelengths that are long against the original context and
    leaves the short ones, with a linear blend of the two frequencies in between."""
    f = float(rot["base"]) ** (-2.0 * np.arange(rot["dims"] // 2) / rot["dims"])
    s = rot.get("scaling")
    if not s or fault == "no_scaling":
        return f
    wavelength = 2.0 * np.pi / f
    out = []
    for fi, l in zip(f, wavelength):
        if l < s["original"] / s["high"]:
            out.append(fi)
        elif l > s["original"] / s["low"]:
            out.append(fi / s["factor"])
        else:
            t = (s["original"] / l - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - t) * fi / s["factor"] + t * fi)
    return np.array(out)


def rotate(x, pos, rot, fault=""):
    """The first rot.dims entries of the last axis, in neighbouring pairs; x [T, ..., d], pos [T]."""
    n = rot["dims"]
    a = pos[:, None] * frequencies(rot, fault)
    a = a.reshape(a.shape[:1] + (1,) * (x.ndim - 2) + a.shape[1:])
    y = x.copy()
    if fault == "half_layout":
        u, v = x[..., :n // 2], x[..., n // 2:n]
        y[..., :n // 2], y[..., n // 2:n] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
        return y
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y[..., 0:n:2], y[..., 1:n:2] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return y


def softmax_rows(s, seen):
    s = np.where(seen, s, -np.inf)
    e = np.exp(s - s.max(axis=1, keepdims=True))
    return e / e.sum(axis=1, keepdims=True)


def visible(T, size=None, fault=""):
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    size = (size or T) + {"window_plus": 1, "window_minus": -1}.get(fault, 0)
    return (d >= 0) & (d < size)


def latent_attention(h, W, p, c, eps, fault="", cache=None):
    """Attention whose keys and values are linear in one normed latent per position, beside one rotated key part that all
    heads share; optionally over a sliding window.  h [T, width] -> [T, width]."""
    T, H, nd, rd, vd, R = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    pos = np.arange(T).astype(h.dtype)
    q = (h @ W[p + "q"].T).reshape(T, H, nd + rd)
    low = h @ W[p + "dkv"].T
    latent, shared = low[:, :R], low[:, R:]
    if fault != "no_latent_norm":
        latent = rms(latent, eps)
    latent = latent * W[p + "dkv.norm"]
    qn, qr = q[..., :nd], rotate(q[..., nd:], pos, c["rot"], fault)
    kr = shared if fault == "shared_key_unrotated" else rotate(shared, pos, c["rot"], fault)
    if cache is not None:
        latent, kr = latent.astype(cache).astype(h.dtype), kr.astype(cache).astype(h.dtype)
    kn = (latent @ W[p + "uk"].T).reshape(T, H, nd)
    v = (latent @ W[p + "uv"].T).reshape(T, H, vd)
    seen = visible(T, (c.get("mask") or {}).get("size"), fault)
    out = np.zeros((T, H, vd), h.dtype)
    for a in range(H):
        s = qn[:, a] @ kn[:, a].T
        if fault != "no_rotated_part":
            s = s + qr[:, a] @ kr.T
        out[:, a] = softmax_rows(s * c["scale"], seen) @ v[:, a]
    return out.reshape(T, H * vd) @ W[p + "o"].T


def difference_factor(W, p, diff):
    return np.exp(np.sum(W[p + "lq1"] * W[p + "lk1"])) - np.exp(np.sum(W[p + "lq2"] * W[p + "lk2"])) + diff


def differential_attention(h, W, p, c, eps, fault="", cache=None):
    """Two causal softmax maps per head over the same values, the second subtracted; per-head norm; a gate on every
    element of the concatenated heads."""
    T, H, G, d, vd, diff = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["diff"]
    pos = np.arange(T).astype(h.dtype)
    q = rotate((h @ W[p + "q"].T).reshape(T, H, 2, d), pos, c["rot"], fault)
    k = rotate((h @ W[p + "k"].T).reshape(T, G, 2, d), pos, c["rot"], fault)
    v = (h @ W[p + "v"].T).reshape(T, G, vd)
    if cache is not None:
        k, v = k.astype(cache).astype(h.dtype), v.astype(cache).astype(h.dtype)
    lam = 0.0 if fault == "one_map" else difference_factor(W, p, diff)
    seen = visible(T)
    out = np.zeros((T, H, vd), h.dtype)
    for a in range(H):
        g = a % G if fault == "heads_interleaved" else a // (H // G)
        maps = [softmax_rows(q[:, a, m] @ k[:, g, m].T * c["scale"], seen) @ v[:, g] for m in (0, 1)]
        o = maps[0] - lam * maps[1]
        if fault != "no_head_norm":
            o = rms(o, eps)
        out[:, a] = o * (1.0 - diff)
    out = out.reshape(T, H * vd)
    if fault != "no_gate":
        out = out * sigmoid(h @ W[p + "g"].T)
    return out @ W[p + "o"].T


def lightning(h, W, p, c, eps, fault="", state=None):
    """Linear attention with one constant decay per head.  `state` [heads, dim, vdim] is updated in place when given."""
    T, H, d, vd = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = silu(h @ W[p + "q"].T).reshape(T, H, d)
    k = silu(h @ W[p + "k"].T).reshape(T, H, d)
    v = silu(h @ W[p + "v"].T).reshape(T, H, vd)
    decay = np.array(c["decay"], h.dtype)[:, None, None]
    S = np.zeros((H, d, vd), h.dtype) if state is None else state
    out = np.zeros((T, H, vd), h.dtype)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        if fault == "decay_after":
            S[:] = decay * (S + kv)
        elif fault == "no_decay":
            S[:] = S + kv
        else:
            S[:] = decay * S + kv
        out[t] = np.einsum("hd,hdv->hv", q[t], S)
    out = rms(out, eps).reshape(T, H * vd) if fault == "norm_per_head" else rms(out.reshape(T, H * vd), eps)
    out = out * W[p + "norm"]
    if fault != "no_gate":
        out = out * sigmoid(h @ W[p + "g"].T)
    return out @ W[p + "o"].T


def gated_ffn(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def token_side(x, W, p, tokens, layer, dim, eps, fault=""):
    """What a layer adds for the tokens themselves: a slice of a second embedding, gated by x."""
    part = 0 if fault == "first_part" else layer
    e = W["side.embed"][np.asarray(tokens)][:, part * dim:(part + 1) * dim]
    y = (gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T
    return rms(y, eps) * W[p + "side.norm"]


MIXERS = {"latent_attention": latent_attention, "attention": differential_attention}


def mixer(h, W, p, L, eps, fault="", cache=None):
    if L["type"] == "lightning":
        return lightning(h, W, p, L["mixer"], eps, fault)
    return MIXERS[L["type"]](h, W, p, L["mixer"], eps, fault, cache)


def layer_runs(cfg, fault=""):
    """(layer, number of the pass it begins or None) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(1 if fault == "one_pass" else loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, W, tokens, fault="", taps=None, cache=None):
    """Logits [T, vocab] of a whole sequence.  `taps`, a list, receives the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)]
    norm = lambda v, name: layer_norm(v, W[name], W[name + ".b"], eps, fault)
    for i, step in layer_runs(cfg, fault):
        L, p = cfg["layers"][i], "l%d." % i
        if step is not None and fault != "no_step":
            x = x + W["loop.step"][0 if fault == "first_step" else step]
        x = x + norm(mixer(norm(x, p + "norm1"), W, p + "mix.", L, eps, fault, cache), p + "norm1b")
        if L.get("mlp"):
            x = x + norm(gated_ffn(norm(x, p + "norm2"), W, p + "mlp."), p + "norm2b")
        if cfg.get("token_side") and fault != "no_side":
            x = x + token_side(x, W, p, tokens, i, cfg["token_side"]["dim"], eps, fault)
        if taps is not None:
            taps.append(x.copy())
    return norm(x, "final.norm") @ W["embed"].T


def greedy(cfg, W, prompt, steps):
    """`steps` tokens after the prompt, each the arg-max of the logits (lowest id on ties); also the smallest gap
    between the two best logits that any of the choices rested on."""
    ids, gap = list(prompt), np.inf
    for _ in range(steps):
        lg = forward(cfg, W, ids)[-1]
        top = np.sort(lg)[-2:]
        gap = min(gap, top[1] - top[0])
        ids.append(int(np.argmax(lg)))
    return ids[len(prompt):], gap
