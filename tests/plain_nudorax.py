"""A plain, slow Nudorax in 64-bit numpy: one function per mechanism, whole sequences only.

It shares nothing with the engine: no kernels, no cache, no step function. A sequence goes in whole and the logits of
every position come out; the recurrence is a Python loop over the tokens, every attention row is worked out by itself
from the keys it may see. `w` maps tensor names to 64-bit arrays, `cfg` is the parsed config.json.

Notation. T tokens, E the model's width, n(v) = v / sqrt(mean(v^2) + eps),
N(v) = (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps). The stream starts as embed[token] * c; a layer is
x <- x + N(mixer(x)) w1, then x <- x + N(ff(x)) w2 where the layer has a feed-forward (both sublayers read the stream
as it is); the logits are s tanh(embed (N(x) w_final) / s).
"""
from __future__ import annotations

import math

import numpy as np

ROUND = None  # a function that rounds an array to the engine's 16-bit format, or None: exact


def mm(a, W):
    """a W^T; with `ROUND` set, `a` is rounded first, as a 16-bit engine rounds what enters a contraction."""
    return (ROUND(a) if ROUND is not None else a) @ W.T


def rms(v, eps):
    return v / np.sqrt(np.mean(v * v, axis=-1, keepdims=True) + eps)


def layer_norm(v, weight, eps):
    d = v - np.mean(v, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * weight


def sigmoid(v):
    return 1.0 / (1.0 + np.exp(-v))


def silu(v):
    return v * sigmoid(v)


# ----------------------------------------------------------------------------------------------- rotation
def frequencies(rot):
    """The dims/2 angular frequencies base^(-2i/dims). With `scaling`: a wave of length l = 2 pi / f is kept where l is
    below original / high, slowed down `factor` times where it is above original / low, and blended in between."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    sc = rot.get("scaling")
    if not sc:
        return f
    factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for fi in f:
        wave = 2.0 * math.pi / fi
        if wave < original / high:
            out.append(fi)
        elif wave > original / low:
            out.append(fi / factor)
        else:
            s = (original / wave - low) / (high - low)
            out.append((1.0 - s) * fi / factor + s * fi)
    return np.array(out)


def rotate_half(v, rot):
    """Entry i of the first `dims` entries turns together with entry i + dims/2; the rest pass. v: [T, heads, d]."""
    f = frequencies(rot)
    half = int(rot["dims"]) // 2
    out = v.copy()
    for p in range(v.shape[0]):
        for i in range(half):
            c, s = math.cos(p * f[i]), math.sin(p * f[i])
            lo, hi = v[p, :, i].copy(), v[p, :, i + half].copy()
            out[p, :, i] = lo * c - hi * s
            out[p, :, i + half] = hi * c + lo * s
    return out


# ----------------------------------------------------------------------------------------------- mixers
def sink_softmax(s, sink):
    """Weights of the scores s when the denominator holds one more term exp(sink) that no value belongs to."""
    top = max(float(s.max()), sink)
    e = np.exp(s - top)
    return e / (math.exp(sink - top) + e.sum())


def window_attention(h, w, p, m, eps):
    """Softmax attention over the last `mask.size` positions, oneself included. Queries and keys are normed over the
    whole projection, all heads at once, then turned by position; the denominator holds exp(sink) of the head."""
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    G = int(m.get("kv_heads") or H)
    dv = int(m.get("vdim") or d)
    q = (rms(mm(h, w[p + "q"]), eps) * w[p + "q.norm"]).reshape(T, H, d)
    k = (rms(mm(h, w[p + "k"]), eps) * w[p + "k.norm"]).reshape(T, G, d)
    v = mm(h, w[p + "v"]).reshape(T, G, dv)
    if m.get("rot"):
        q, k = rotate_half(q, m["rot"]), rotate_half(k, m["rot"])
    if ROUND is not None:
        q, k, v = ROUND(q), ROUND(k), ROUND(v)  # 16-bit queries; the cache holds 16-bit keys and values
    size = int(m["mask"]["size"]) if m.get("mask") else T
    out = np.zeros((T, H, dv))
    for t in range(T):
        lo = max(0, t - size + 1)
        for a in range(H):
            kv = a // (H // G)
            s = (k[lo:t + 1, kv] @ q[t, a]) * float(m["scale"])
            out[t, a] = sink_softmax(s, float(w[p + "sink"][a])) @ v[lo:t + 1, kv]
    return mm(out.reshape(T, H * dv), w[p + "o"])


def lightning(h, w, p, m, eps):
    """Linear attention with one fixed decay per head behind silu: per head S [dim, vdim] from zero,
    S <- decay S + k v^T, o = S^T q; the concatenated heads are normed together, gated and projected."""
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    dv = int(m.get("vdim") or d)
    q = silu(mm(h, w[p + "q"])).reshape(T, H, d)
    k = silu(mm(h, w[p + "k"])).reshape(T, H, d)
    v = silu(mm(h, w[p + "v"])).reshape(T, H, dv)
    if ROUND is not None:
        q, k, v = ROUND(q), ROUND(k), ROUND(v)
    out = np.zeros((T, H, dv))
    for a in range(H):
        S = np.zeros((d, dv))
        for t in range(T):
            S = float(m["decay"][a]) * S + np.outer(k[t, a], v[t, a])
            out[t, a] = S.T @ q[t, a]
    out = rms(out.reshape(T, H * dv), eps) * w[p + "norm"] * sigmoid(mm(h, w[p + "g"]))
    return mm(out, w[p + "o"])


def parallel(h, w, p, m, eps):
    return (float(m["left_scale"]) * window_attention(h, w, p + "left.", m["left"], eps)
            + float(m["right_scale"]) * lightning(h, w, p + "right.", m["right"], eps))


# ----------------------------------------------------------------------------------------------- feed-forwards
def capped_unit(f, w, p, limit):
    g = np.minimum(mm(f, w[p + "gate"]), limit)
    u = np.clip(mm(f, w[p + "up"]), -limit, limit)
    return mm(g * sigmoid(1.702 * g) * (u + 1.0), w[p + "down"])


def chosen_experts(s, router):
    """The `top` largest scores (the lower number on a tie) among the experts of the best groups: equal runs of
    neighbours, a run's score the sum of its two largest."""
    allowed = set(range(len(s)))
    groups = router.get("groups")
    if groups:
        size = len(s) // int(groups["count"])
        score = [sum(sorted(s[g * size:(g + 1) * size])[-2:]) for g in range(int(groups["count"]))]
        best = sorted(range(len(score)), key=lambda g: (-score[g], g))[:int(groups["keep"])]
        allowed = {e for g in best for e in range(g * size, (g + 1) * size)}
    return sorted(allowed, key=lambda e: (-s[e], e))[:int(router["top"])]


def routed_ff(f, w, p, mlp):
    """Each token's chosen experts weighted by their sigmoid scores times a constant, plus the shared expert weighted
    by the sigmoid of one number per token."""
    router, limit = mlp["router"], float(mlp["expert"]["limit"])
    scores = sigmoid(mm(f, w[p + "router"]))
    scale = float(router.get("scale", 1.0))
    out = np.zeros_like(f)
    for t in range(f.shape[0]):
        for e in sorted(chosen_experts(scores[t], router)):
            out[t] += scores[t, e] * scale * capped_unit(f[t:t + 1], w, f"{p}e{e}.", limit)[0]
    if mlp.get("shared"):
        gate = sigmoid(mm(f, w[p + "shared.sg"]))  # [T, 1]
        out += gate * capped_unit(f, w, p + "shared.", float(mlp["shared"]["limit"]))
    return out


# ----------------------------------------------------------------------------------------------- the model
def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence. `layers_out`: a list that receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][np.asarray(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + layer_norm(parallel(x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + layer_norm(routed_ff(x, w, p + "mlp.", layer["mlp"]), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    logits = mm(layer_norm(x, w["final.norm"], eps), w["embed"])
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(logits / cap) if cap else logits
