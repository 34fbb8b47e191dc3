"""Plain, slow implementation of the Novunex decoder in numpy: whole sequences, no cache, one function per mechanism.  It shares
no code with the engine: it reads config.json keys itself and walks tokens, heads and experts with ordinary loops where the
engine has kernels.

A Novunex layer's sublayers read the stream itself, and only what they return is normed:

    x <- x + N1(mixer(x));    x <- x + N2(ff(x)),      N(y) = y / rms(y) * w

The mixer is grouped-query softmax attention with rotation, in two forms: "attention" norms every q and k head over its own
numbers and adds one to the softmax's denominator; "attention_2" norms the whole q and k projections, scales the rotation's
frequencies by wavelength, and may read an earlier layer's keys and values.  ff is a mixture of small feed-forwards of which
some are the identity, with a shared one beside it, or absent.

All arithmetic is float64; tensors come as a dict of arrays.
"""

from __future__ import annotations

import numpy as np


def rms_norm(x, weight, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * weight


def frequencies(rot):
    """One angle per position and pair; with ``scaling`` long wavelengths are stretched by its factor, short ones kept, and those
    between blended by where original / wavelength lies between low and high."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wave = 2 * np.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                share = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = share * f + (1 - share) * f / s["factor"]
        out.append(f)
    return np.array(out)


def rotate(x, rot):
    """x [T, heads, dim]: dimension i turns with dimension i + dims / 2 by position times frequency; the rest stay."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    angle = np.arange(x.shape[0])[:, None, None] * frequencies(rot)
    u, v = x[..., :half], x[..., half : 2 * half]
    return np.concatenate([u * np.cos(angle) - v * np.sin(angle), v * np.cos(angle) + u * np.sin(angle), x[..., 2 * half :]], -1)


def normed_heads(y, heads, weight, eps, per_head):
    """A q or k projection [T, heads * dim] as [T, heads, dim], normed head by head or as a whole."""
    T = y.shape[0]
    if per_head:
        return rms_norm(y.reshape(T, heads, -1), weight, eps)
    return rms_norm(y, weight, eps).reshape(T, heads, -1)


def keys_and_values(h, w, px, m, eps, per_head):
    k = rotate(normed_heads(h @ w[px + "k"].T, m["kv_heads"], w[px + "k.norm"], eps, per_head), m.get("rot"))
    return k, (h @ w[px + "v"].T).reshape(h.shape[0], m["kv_heads"], m["vdim"])


def softmax_weights(s, one_more):
    """exp(s) over its sum — plus one, with ``one_more``."""
    top = max(s.max(), 0.0) if one_more else s.max()
    p = np.exp(s - top)
    return p / (p.sum() + (np.exp(-top) if one_more else 0.0))


def attention(h, w, px, m, eps, per_head, one_more, keys, values):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rotate(normed_heads(h @ w[px + "q"].T, H, w[px + "q.norm"], eps, per_head), m.get("rot"))
    out = np.zeros((T, H, m["vdim"]))
    for a in range(H):
        g = a // (H // G)
        for t in range(T):
            out[t, a] = softmax_weights((keys[: t + 1, g] @ q[t, a]) * m["scale"], one_more) @ values[: t + 1, g]
    return out.reshape(T, -1) @ w[px + "o"].T


def squared_relu(h, w, px):
    return np.maximum(h @ w[px + "up"].T, 0) ** 2 @ w[px + "down"].T


def route(h, w, px, top):
    """Which experts a token uses, best first, and with what weights: [T, top] each.  A correction steers the choice alone."""
    z = h @ w[px + "router"].T
    s = np.exp(z - z.max(1, keepdims=True))
    s = s / s.sum(1, keepdims=True)
    ids = np.argsort(-(s + w[px + "correction"]), axis=1, kind="stable")[:, :top]
    return ids, np.take_along_axis(s, ids, 1)


def feed_forward(h, w, px, mlp):
    r = mlp["router"]
    ids, weights = route(h, w, px, r["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(ids[t], weights[t]):
            out[t] += g * (squared_relu(h[t : t + 1], w, f"{px}e{e}.")[0] if e < r["experts"] else h[t])
    return out + (squared_relu(h, w, px + "shared.") if mlp.get("shared") else 0.0)


def forward(cfg, w, tokens, trace=None):
    """Logits [T, vocab] of one sequence; ``trace`` (a list) collects the stream after every layer."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    cached = {}  # layer -> its keys and values
    for i, entry in enumerate(cfg["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        per_head = one_more = entry["type"] == "attention"
        owner = i if m.get("kv_from") is None else m["kv_from"]
        if owner == i:
            cached[i] = keys_and_values(x, w, p + "mix.", m, eps, per_head)
        x = x + rms_norm(attention(x, w, p + "mix.", m, eps, per_head, one_more, *cached[owner]), w[p + "norm1"], eps)
        if entry.get("mlp") is not None:
            x = x + rms_norm(feed_forward(x, w, p + "mlp.", entry["mlp"]), w[p + "norm2"], eps)
        if trace is not None:
            trace.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, w, prompt, new_tokens):
    tokens = list(prompt)
    for _ in range(new_tokens):
        tokens.append(int(np.argmax(forward(cfg, w, tokens)[-1])))
    return tokens[len(prompt):]
