"""A plain, slow Pafutar in 64-bit numpy: one function per mechanism, whole sequences only.

It shares nothing with the engine: no kernels, no cache, no step function. A sequence goes in whole and the logits of
every position come out; every attention row is worked out by itself from the keys it may see. `w` maps tensor names to
64-bit arrays, `cfg` is the parsed config.json.

Notation. T tokens, n(v) = v / sqrt(mean(v^2) + eps), a the configuration's `postln_alpha`. The stream starts as
embed[token] * c + pos[t]; a layer is x <- n(a x + s1 * mixer(mix(x))) * w1, where mix blends every row with the one
before it, then x <- n(a x + s2 * ff(x)) * w2 where the layer has a feed-forward; the logits are head (n(x) * w_final).
"""
from __future__ import annotations

import numpy as np

ROUND = None  # a function that rounds an array to the engine's 16-bit format, or None: exact


def rounded(a):
    return ROUND(a) if ROUND is not None else a


def mm(a, W):
    """a W^T; with `ROUND` set, `a` is rounded first, as a 16-bit engine rounds what enters a contraction."""
    return rounded(a) @ W.T


def rms(v, eps):
    return v / np.sqrt(np.mean(v * v, axis=-1, keepdims=True) + eps)


def sigmoid(v):
    return 1.0 / (1.0 + np.exp(-v))


# ----------------------------------------------------------------------------------------------- around the sublayers
def embed(cfg, w, tokens):
    c = float((cfg.get("embedding") or {}).get("scale", 1.0))
    x = w["embed"][np.asarray(tokens)] * c
    return x + w["pos"][:len(tokens)]


def shift(x, mix):
    """Row t is moved towards row t - 1 (nothing stands before row 0) by the share `mix`, per channel."""
    before = np.vstack([np.zeros((1, x.shape[1])), x[:-1]])
    return x + (before - x) * mix


def sum_norm(x, y, alpha, scale, weight, eps):
    return rms(alpha * x + scale * y, eps) * weight


# ----------------------------------------------------------------------------------------------- attention
def visible(t, mask):
    """The positions row t sees: the last `size` ones, itself included, and the first `keep_first` of the sequence."""
    if not mask:
        return np.arange(t + 1)
    size, keep = int(mask["size"]), int(mask.get("keep_first") or 0)
    return np.array([j for j in range(t + 1) if t - j < size or j < keep])


def slopes(heads):
    return [2.0 ** (-8.0 * (a + 1) / heads) for a in range(heads)]


def attention(h, w, p, m, eps):
    """Softmax attention over a window and the first tokens. Queries and keys are divided by their root mean square per
    head; a score is scaled, times the head's factor, less the head's slope times the distance. The values are the keys
    as projected. The heads pass a sigmoid gate, one number per value, before the output projection."""
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    G = int(m.get("kv_heads") or H)
    scale = float(m["scale"]) if m.get("scale") is not None else d ** -0.5
    q = rounded(mm(h, w[p + "q"]) + w[p + "q.b"]).reshape(T, H, d)
    v = rounded(mm(h, w[p + "k"]) + w[p + "k.b"]).reshape(T, G, d)
    q, k = rounded(rms(q, eps)), rounded(rms(v, eps))
    temp, slope = w[p + "temp"], slopes(H)
    out = np.zeros((T, H, d))
    for t in range(T):
        js = visible(t, m.get("mask"))
        for a in range(H):
            g = a // (H // G)
            s = (k[js, g] @ q[t, a]) * scale * temp[a] - slope[a] * (t - js)
            e = np.exp(s - s.max())
            out[t, a] = rounded(e / e.sum()) @ v[js, g]
    gate = sigmoid(rounded(mm(h, w[p + "g"])))
    return mm(out.reshape(T, H * d) * gate, w[p + "o"])


# ----------------------------------------------------------------------------------------------- feed-forward
def relu2_ff(f, w, p):
    u = np.maximum(mm(f, w[p + "up"]), 0.0)
    return mm(u * u, w[p + "down"])


# ----------------------------------------------------------------------------------------------- the model
def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence. `layers_out`: a list that receives the stream after every layer run."""
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    x = embed(cfg, w, tokens)
    for i, layer in enumerate(cfg["layers"]):
        j = i
        while cfg["layers"][j].get("weights_of") is not None:
            j = cfg["layers"][j]["weights_of"]
        x = run_layer(x, w, f"l{j}.", layer, alpha, eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return mm(rms(x, eps) * w["final.norm"], w["head"])


def run_layer(x, w, p, layer, alpha, eps):
    y = attention(shift(x, w[p + "shift"]), w, p + "mix.", layer["mixer"], eps)
    x = sum_norm(x, y, alpha, w[p + "ls1"], w[p + "norm1"], eps)
    if layer.get("mlp"):
        x = sum_norm(x, relu2_ff(x, w, p + "mlp."), alpha, w[p + "ls2"], w[p + "norm2"], eps)
    return x
