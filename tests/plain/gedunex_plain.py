"""Plain, slow implementation of the Gedunex decoder in numpy: whole sequences, no cache, one function per mechanism.  It
shares no code with the engine: it reads config.json keys itself and walks tokens and keys with ordinary loops where the
engine has kernels.

A Gedunex layer reads the stream once, behind one norm, and adds both of its sublayers' outputs to it:

    h = N(x);    x <- x + (mixer(h) + ff(h)),      N(x) = x / rms(x) * w

The mixer is a matrix memory with exponential gates ("mlstm") or windowed softmax attention without rotation ("attention":
norm over the whole q and k projections, a query temperature that grows with the position, soft-capped scores, a penalty per
head that grows with the distance, a sink per head, values mixed with an earlier layer's).  ff is a dense gated
feed-forward, a routed mixture of small ones, or absent.  The embedding is scaled and a sinusoidal position vector added.

All arithmetic is float64; tensors come as a dict of arrays.
"""

from __future__ import annotations

import numpy as np


def rms_unit(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def sigmoid(z):
    return np.where(z >= 0, 1 / (1 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return np.minimum(z, 0) - np.log1p(np.exp(-np.abs(z)))


def position_vectors(T, width):
    """[T, width]: sines in the even places, cosines in the odd ones, the pair's frequency 10000^(-2i/width)."""
    out = np.zeros((T, width))
    for c in range(width):
        angle = np.arange(T) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = np.sin(angle) if c % 2 == 0 else np.cos(angle)
    return out


def embed(w, cfg, tokens):
    x = w["embed"][np.asarray(tokens)] * (cfg.get("embedding") or {}).get("scale", 1.0)
    return x + position_vectors(len(tokens), cfg["width"])


def matrix_memory(h, w, px, m, eps):
    """Per head a matrix S and a vector n that decay by a gate of the token's own, with gates kept as logarithms and everything
    divided by exp(running maximum)."""
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[px + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[px + "k"].T).reshape(T, H, d)
    v = (h @ w[px + "v"].T).reshape(T, H, dv)
    log_in = cap * np.tanh((h @ w[px + "i"].T + w[px + "i.b"]) / cap)
    log_forget = log_sigmoid(cap * np.tanh((h @ w[px + "f"].T + w[px + "f.b"]) / cap))
    out = np.zeros((T, H, dv))
    for a in range(H):
        S, n, top = np.zeros((d, dv)), np.zeros(d), 0.0
        for t in range(T):
            new = max(log_forget[t, a] + top, log_in[t, a])
            keep, take = np.exp(log_forget[t, a] + top - new), np.exp(log_in[t, a] - new)
            S = keep * S + take * np.outer(k[t, a], v[t, a])
            n = keep * n + take * k[t, a]
            top = new
            out[t, a] = S.T @ q[t, a] / (max(abs(n @ q[t, a]), np.exp(-top)) + 1e-6)
    y = rms_unit(out, eps).reshape(T, H * dv) * w[px + "norm"] * sigmoid(h @ w[px + "g"].T)
    return y @ w[px + "o"].T


def slopes(H):
    return [2.0 ** (-8.0 * (a + 1) / H) for a in range(H)]


def temperature(T, q_temp):
    if not q_temp:
        return np.ones(T)
    p = np.arange(T)
    return 1 + q_temp["coef"] * np.log(np.floor((p + 1) / q_temp["every"]) + 1)


def attention(h, w, px, m, eps, first_values):
    """``first_values``: None in a layer whose values stay as they are, else the values of the first mixing layer.  Returns the
    output and this layer's values before mixing."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit(h @ w[px + "q"].T + w[px + "q.b"], eps) * w[px + "q.norm"]
    k = rms_unit(h @ w[px + "k"].T + w[px + "k.b"], eps) * w[px + "k.norm"]
    own = h @ w[px + "v"].T + w[px + "v.b"]
    v = own
    if first_values is not None:
        lam = float(w[px + "vmix"])
        v = (1 - lam) * own + lam * first_values
    q = (q * temperature(T, m.get("q_temp"))[:, None]).reshape(T, H, d)
    k, v = k.reshape(T, G, d), v.reshape(T, G, dv)
    size = (m.get("mask") or {}).get("size")
    out = np.zeros((T, H, dv))
    for a in range(H):
        g, slope, sink = a // (H // G), slopes(H)[a], w[px + "sink"][a]
        for t in range(T):
            first = 0 if size is None else max(0, t - size + 1)
            s = (k[first : t + 1, g] @ q[t, a]) * m["scale"]
            if m.get("softcap"):
                s = m["softcap"] * np.tanh(s / m["softcap"])
            s = s - slope * (t - np.arange(first, t + 1))
            top = max(s.max(), sink)
            p = np.exp(s - top)
            out[t, a] = (p / (p.sum() + np.exp(sink - top))) @ v[first : t + 1, g]
    return out.reshape(T, H * dv) @ w[px + "o"].T, own


def gated(h, w, px):
    return (silu(h @ w[px + "gate"].T) * (h @ w[px + "up"].T)) @ w[px + "down"].T


def route(h, w, px, r):
    """Which experts a token uses and with what weights: [T, top] indices and weights."""
    z = h @ w[px + "router"].T + w[px + "router.b"]
    ids = np.argsort(-z, axis=1, kind="stable")[:, : r["top"]]
    picked = np.take_along_axis(z, ids, 1)
    p = np.exp(picked - picked.max(1, keepdims=True))
    return ids, p / p.sum(1, keepdims=True)


def feed_forward(h, w, px, mlp):
    if mlp["kind"] == "dense":
        return gated(h, w, px)
    ids, weights = route(h, w, px, mlp["router"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(ids[t], weights[t]):
            out[t] += g * gated(h[t : t + 1], w, f"{px}e{e}.")[0]
    return out


def forward(cfg, w, tokens, trace=None):
    """Logits [T, vocab] of one sequence; ``trace`` (a list) collects the stream after every layer."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = embed(w, cfg, tokens)
    first_values = None  # of the first layer that mixes values
    for i, entry in enumerate(cfg["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        h = rms_unit(x, eps) * w[p + "norm1"]
        if entry["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            delta, own = attention(h, w, p + "mix.", m, eps, first_values if mixes else None)
            if mixes and first_values is None:
                first_values = own
        else:
            delta = matrix_memory(h, w, p + "mix.", m, eps)
        if entry.get("mlp") is not None:
            delta = delta + feed_forward(h, w, p + "mlp.", entry["mlp"])
        x = x + delta
        if trace is not None:
            trace.append(x.copy())
    return (rms_unit(x, eps) * w["final.norm"]) @ w["head"].T


def greedy(cfg, w, prompt, new_tokens):
    tokens = list(prompt)
    for _ in range(new_tokens):
        tokens.append(int(np.argmax(forward(cfg, w, tokens)[-1])))
    return tokens[len(prompt):]
