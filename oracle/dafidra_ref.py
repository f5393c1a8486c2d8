"""A plain numpy restatement of the Dafidra decoder (TEST INFRASTRUCTURE ONLY).

One function per mechanism, written for one sequence at a time, token by token where the mechanism is a
recurrence and over the whole sequence where it is not.  Nothing here is shared with the product: no kernel,
no loader, no cache.  Weights are a dict name -> float array (matrices [out, in]); the configuration is the
dict a config.json holds.  All arithmetic is float64 unless `ft` says otherwise, so that a comparison measures
the product's rounding and not this file's.

`fault` names a deliberate mistake to make in one mechanism; tests use it to show that their inputs would
expose that mistake.
"""
import numpy as np


def rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_around_zero(x, w, eps):
    """RMS norm whose weight is stored minus one."""
    return rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z / (1.0 + np.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def log_sigmoid(z):
    return -(np.maximum(-z, 0.0) + np.log1p(np.exp(-np.abs(z))))


def query_temperature(pos, every, coef):
    return 1.0 + coef * np.log(np.floor((pos + 1.0) / every) + 1.0)


def head_slopes(heads):
    return 2.0 ** (-8.0 * (np.arange(heads) + 1.0) / heads)


def attention(h, W, p, c, eps, fault="", cache=None):
    """Windowed softmax attention: whole-projection q/k norm, temperature on q, linear distance bias, a sink in the
    denominator, one output gate per head.  h [T, width] -> [T, width].  `cache` (a numpy type) rounds keys and values to
    what a cache of that type holds."""
    T = h.shape[0]
    H, G, dim, vdim = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = h @ W[p + "q"].T, h @ W[p + "k"].T, h @ W[p + "v"].T
    if fault == "norm_per_head":
        q = rms(q.reshape(T, H, dim), eps).reshape(T, -1) * W[p + "q.norm"]
    else:
        q = norm_plain(q, W[p + "q.norm"], eps)
    k = norm_plain(k, W[p + "k.norm"], eps)
    if cache is not None:
        k, v = k.astype(cache).astype(np.float64), v.astype(cache).astype(np.float64)
    pos = np.arange(T)
    if fault != "no_temperature":
        q = q * query_temperature(pos, c["q_temp"]["every"], c["q_temp"]["coef"])[:, None]
    q, k, v = q.reshape(T, H, dim), k.reshape(T, G, dim), v.reshape(T, G, vdim)
    window = (c.get("mask") or {}).get("size") or T
    window += {"window_plus": 1, "window_minus": -1}.get(fault, 0)
    slopes = head_slopes(H)
    dist = pos[:, None] - pos[None, :]
    seen = (dist >= 0) & (dist < window)
    gate = sigmoid(h @ W[p + "g"].T)
    out = np.zeros((T, H, vdim))
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * c["scale"]
        if fault != "no_bias":
            s = s - slopes[a] * dist
        s = np.where(seen, s, -np.inf)
        sink = W[p + "sink"][a]
        m = s.max(axis=1)
        if fault != "no_sink":
            m = np.maximum(m, sink)
        e = np.exp(s - m[:, None])
        den = e.sum(axis=1)
        if fault != "no_sink":
            den = den + np.exp(sink - m)
        out[:, a] = (e @ v[:, g]) / den[:, None]
        if fault != "no_gate":
            out[:, a] *= gate[:, a:a + 1]
    return out.reshape(T, H * vdim) @ W[p + "o"].T


def matrix_memory(h, W, p, c, eps, fault="", state=None):
    """Matrix memory with exponential input and sigmoid forget gates, a running maximum that starts at zero.
    `state` (S [heads, dim, vdim], n [heads, dim], m [heads]) is updated in place when given."""
    T = h.shape[0]
    H, dim, vdim, cap = c["heads"], c["dim"], c["vdim"], c["gate_cap"]
    q = (h @ W[p + "q"].T).reshape(T, H, dim) * dim ** -0.5
    k = (h @ W[p + "k"].T).reshape(T, H, dim)
    v = (h @ W[p + "v"].T).reshape(T, H, vdim)
    gi = cap * np.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    gf = log_sigmoid(cap * np.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap))
    if state is None:
        state = (np.zeros((H, dim, vdim)), np.zeros((H, dim)), np.full(H, -np.inf if fault == "max_from_minus_inf" else 0.0))
    S, n, m = state
    out = np.zeros((T, H, vdim))
    for t in range(T):
        mt = np.maximum(gf[t] + m, gi[t])
        fa, ia = np.exp(gf[t] + m - mt), np.exp(gi[t] - mt)
        S[:] = fa[:, None, None] * S + ia[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n[:] = fa[:, None] * n + ia[:, None] * k[t]
        m[:] = mt
        num = np.einsum("hd,hdv->hv", q[t], S)
        den = np.maximum(np.abs(np.einsum("hd,hd->h", n, q[t])), np.exp(-m)) + 1e-6
        out[t] = num / den[:, None]
    out = rms(out, eps).reshape(T, H * vdim) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)
    return out @ W[p + "o"].T


def parallel_mixer(h, W, p, c, eps, fault="", state=None, cache=None):
    """Both mixers on the same input, each output normed over the width, averaged."""
    a = norm_plain(attention(h, W, p + "left.", c["left"], eps, fault, cache), W[p + "left.out"], eps)
    b = norm_plain(matrix_memory(h, W, p + "right.", c["right"], eps, fault, state), W[p + "right.out"], eps)
    return (a + b) * 0.5


def gated_ffn(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(z, experts, top, groups=None, fault=""):
    """Chosen experts and their weights for one token's router logits: scores are a softmax over all experts, only the
    groups with the largest best scores may be chosen from, the weights are the scores unchanged."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    allowed = np.ones(experts, bool)
    if groups and fault != "no_groups":
        count, keep = groups["count"], groups["keep"]
        best = s.reshape(count, experts // count).max(axis=1)
        kept = np.argsort(-best, kind="stable")[:keep]
        allowed = np.isin(np.arange(experts) // (experts // count), kept)
    ranked = np.argsort(np.where(allowed, -s, np.inf), kind="stable")[:top]
    w = s[ranked]
    if fault == "renormalise":
        w = w / w.sum()
    return ranked, w


def route_margin(z, experts, top, groups=None):
    """How far a token's routing is from another outcome: the smallest relative gap between the scores (of experts, and of
    groups) on either side of a choice."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    margin, allowed = 1.0, np.ones(experts, bool)
    if groups and groups["keep"] < groups["count"]:
        best = s.reshape(groups["count"], -1).max(axis=1)
        r = np.sort(best)[::-1]
        margin = min(margin, (r[groups["keep"] - 1] - r[groups["keep"]]) / r[groups["keep"] - 1])
        kept = np.argsort(-best, kind="stable")[:groups["keep"]]
        allowed = np.isin(np.arange(experts) // (experts // groups["count"]), kept)
    r = np.sort(s[allowed])[::-1]
    if top < len(r):
        margin = min(margin, (r[top - 1] - r[top]) / r[top - 1])
    return margin


def feed_forward(h, W, p, c, fault="", margins=None):
    if c["kind"] == "dense":
        return gated_ffn(h, W, p)
    r = c["router"]
    out = np.zeros_like(h)
    z = h @ W[p + "router"].T
    for t in range(h.shape[0]):
        ids, w = route(z[t], r["experts"], r["top"], r.get("groups"), fault)
        if margins is not None:
            margins.append(route_margin(z[t], r["experts"], r["top"], r.get("groups")))
        for e, we in zip(ids, w):
            out[t] += we * gated_ffn(h[t:t + 1], W, "%se%d." % (p, e))[0]
    return out


def forward(cfg, W, tokens, fault="", taps=None, margins=None, cache=None):
    """Logits [T, vocab] of a whole sequence.  `taps`, a list, receives the residual stream after every layer, `margins`
    the routing margin of every token and layer."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][np.asarray(tokens)]
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % i
        assert L["type"] == "parallel"
        x = x + mult * norm_around_zero(parallel_mixer(x, W, p + "mix.", L["mixer"], eps, fault, cache=cache), W[p + "norm1"], eps)
        if L.get("mlp"):
            x = x + mult * norm_around_zero(feed_forward(x, W, p + "mlp.", L["mlp"], fault, margins), W[p + "norm2"], eps)
        if taps is not None:
            taps.append(x.copy())
    return norm_around_zero(x, W["final.norm"], eps) @ W["head"].T


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
