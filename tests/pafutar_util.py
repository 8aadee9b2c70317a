"""Small Pafutar configurations with weights that exercise every mechanism, for the engine and for the plain implementation
alike (the same values, bfloat16-rounded, as a folder and as 64-bit arrays)."""
from __future__ import annotations

import copy

import numpy as np
import torch

import plain_pafutar
from bananex_util import bf16_round, plain_weights, random_tokens, write_model  # noqa: F401  (shared helpers)


def attn(heads=4, kv_heads=2, dim=16, scale=0.5, window=13, keep=3, vdim=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim}
    if scale is not None:
        m["scale"] = scale
    if vdim:
        m["vdim"] = dim
    if window is not None:
        m["mask"] = {"size": window, "keep_first": keep}
    return m


def layer(m=None, ff=40, of=None):
    out = {"type": "attention", "mixer": m if m is not None else attn(), "mlp": {"kind": "dense", "ff": ff} if ff else None}
    if of is not None:
        out["weights_of"] = of
    return out


def config(layers, width=60, vocab=199, eps=1e-5, alpha=1.7, scale=3.0, max_positions=700):
    cfg = {"architecture": "Pafutar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
           "max_positions": max_positions, "layers": [copy.deepcopy(l) for l in layers]}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    return cfg


# sizes that differ in every respect: key heads shared or not, one head, windows of one key, inside and across pages and
# 64-key tiles, longer than most prompts and none, no kept keys, a few, a page's worth and more than a tile's, layers without
# a feed-forward, tensors borrowed from the layer before, from a later one and through another borrower, a model with a
# different group of pages per layer, widths that are no multiple of four or eight, alpha 1 and below, embedding rows as stored
CONFIGS = {
    "mix": config([layer(), layer(attn(heads=3, kv_heads=3, dim=8, window=5, keep=1), ff=None), layer(of=0),
                   layer(attn(window=40, keep=9), ff=24), layer(attn(heads=3, kv_heads=3, dim=8, window=5, keep=1), ff=None, of=1),
                   layer(of=2)]),
    "plain": config([layer(attn(heads=2, kv_heads=1, window=None), ff=56), layer(attn(heads=2, kv_heads=1, window=None), ff=56, of=2),
                     layer(attn(heads=2, kv_heads=1, window=None), ff=56), layer(attn(heads=5, kv_heads=1, dim=12, scale=None, window=64, keep=0, vdim=False))],
                    width=48, vocab=131, alpha=1.0, scale=None, max_positions=300),
    "one": config([layer(attn(heads=1, kv_heads=1, dim=32, scale=0.4, window=1, keep=0), ff=7), layer(attn(heads=1, kv_heads=1, dim=20, window=29, keep=70), ff=9),
                   layer(attn(heads=6, kv_heads=2, dim=12, scale=1.2, window=1, keep=1), ff=None)],
                  width=42, vocab=97, eps=1e-6, alpha=0.8, scale=6.5, max_positions=150),
    # (shapes of a kind the tensor-core kernels take in bfloat16)
    "wide": config([layer(attn(heads=6, kv_heads=2, dim=64, scale=0.2, window=37, keep=2), ff=96), layer(attn(heads=2, kv_heads=1, dim=128, scale=None, window=75, keep=66), ff=128),
                    layer(attn(heads=4, kv_heads=4, dim=32, window=200, keep=5), ff=64), layer(attn(heads=16, kv_heads=1, dim=16, window=90, keep=17), ff=None),
                    layer(attn(heads=6, kv_heads=2, dim=64, scale=0.2, window=37, keep=2), ff=96, of=0)],
                   width=96, vocab=257),
    "two": config([layer(attn(heads=2, kv_heads=1, dim=64), ff=64)] * 2 + [layer(attn(heads=2, kv_heads=1, dim=64), ff=64, of=1)], width=64, vocab=89,
                  max_positions=256),
}


def draw(name: str, need, rng) -> np.ndarray:
    """One tensor's values. Matrices N(0, 1/fan_in) so activations stay of order one; norm gains and layer scales 1 + N(0,
    0.2); biases and the heads' factors well away from nothing, negative factors among them; shares of the previous token
    from 0 to 1."""
    shape = tuple(need.shape)
    if name.endswith(".temp"):
        return rng.choice([-1.0, 1.0, 1.0], shape) * rng.uniform(0.4, 2.2, shape)
    if name.endswith(".shift"):
        return rng.uniform(0.0, 1.0, shape)
    if name.endswith(".b"):
        return rng.normal(0.0, 0.5, shape)
    if need.init == "ones":
        return 1.0 + rng.normal(0.0, 0.2, shape)
    if name in ("embed", "pos"):
        return rng.normal(0.0, 1.0, shape)
    return rng.normal(0.0, 1.0, shape) / np.sqrt(shape[-1])


def make_weights(cfg: dict, seed: int) -> dict:
    """name -> bfloat16 tensor for every tensor the model asks for."""
    from cuca_b200.config.registry import build_spec
    from cuca_b200.models.model import Model

    needs = Model(build_spec(cfg), runtime=None).tensor_needs()
    rng = np.random.default_rng(seed)
    return {name: torch.from_numpy(np.asarray(draw(name, need, rng), dtype=np.float32)).to(torch.bfloat16)
            for name, need in sorted(needs.items())}


class Oracle:
    """Whole-sequence logits of the plain implementation, exact and with what enters contractions and caches rounded to
    bfloat16, cached per request (the interface `replay_util.compare` takes)."""

    def __init__(self, cfg: dict, weights: dict):
        self.cfg, self.w = cfg, plain_weights(weights)
        self._cache = {}

    def logits(self, rid: str, tokens: list) -> np.ndarray:
        if rid not in self._cache:
            self._cache[rid] = plain_pafutar.forward(self.cfg, self.w, tokens)
        return self._cache[rid]

    def tolerance(self, dtype: str, requests: dict) -> float:
        """What a replay may differ by, relative to a row's largest logit. 32-bit: a fixed small number. bfloat16: three
        times what rounding alone does to these very requests at its worst, at least 2e-2."""
        if dtype == "float32":
            return 1e-4
        worst = 0.0
        for rid, tokens in requests.items():
            exact = self.logits(rid, tokens)
            plain_pafutar.ROUND = bf16_round
            try:
                rounded = plain_pafutar.forward(self.cfg, self.w, tokens)
            finally:
                plain_pafutar.ROUND = None
            worst = max(worst, float((np.abs(rounded - exact).max(axis=1) / np.abs(exact).max(axis=1)).max()))
        return max(2e-2, 3.0 * worst)


def compare(steps, got, requests, oracle, dtype, tolerance=None):
    import replay_util as ru
    return ru.compare(steps, got, requests, oracle, tolerance or oracle.tolerance(dtype, requests))
