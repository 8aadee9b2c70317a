"""Small Nudorax configurations with weights that exercise every mechanism, for the engine and for the plain
implementation alike (the same values, bfloat16-rounded, as a folder and as 64-bit arrays)."""
from __future__ import annotations

import copy

import numpy as np
import torch

import plain_nudorax
from bananex_util import bf16_round, plain_weights, random_tokens, write_model  # noqa: F401  (shared helpers)
from sutosun_util import compare  # noqa: F401  (the comparison for models with routed layers)

WAVES = {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 60}


def left(heads=4, kv_heads=2, dim=16, vdim=24, scale=None, window=13, base=5000.0, dims=12, scaling=WAVES):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
         "scale": scale if scale is not None else dim ** -0.5}
    if window is not None:
        m["mask"] = {"size": window}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
        if scaling:
            m["rot"]["scaling"] = dict(scaling)
    return m


def right(heads=3, dim=12, vdim=20, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim,
            "decay": list(decay) if decay is not None else [1.0 - 2.0 ** -(1 + 3 * a) for a in range(heads)]}


def mixer(l=None, r=None, ls=0.75, rs=1.25):
    return {"left": l if l is not None else left(), "right": r if r is not None else right(), "left_scale": ls,
            "right_scale": rs}


def moe(ff=24, limit=1.5, experts=6, top=2, groups=(3, 2), scale=1.75, shared=(40, 0.8)):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def config(mixers, mlps, width=60, vocab=199, eps=1e-5, softcap=12.0, scale=1.6):
    cfg = {"architecture": "Nudorax", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "layers": [{"type": "parallel", "mixer": copy.deepcopy(m), "mlp": copy.deepcopy(f)} for m, f in zip(mixers, mlps)]}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    if softcap is not None:
        cfg["logit_softcap"] = softcap
    return cfg


# sizes that differ in every respect: key heads shared or not, one head, values wider and narrower than keys and as wide,
# windows of one key, of a few pages, longer than most prompts and none, rotation of all, part or none of a head with and
# without scaled frequencies, decays from fast to none, layers without a feed-forward, one expert of one, all experts of
# the kept groups chosen, groups of one expert, no groups, no shared expert, a shared expert wider and narrower than the
# others, a side that is subtracted, no cap on the logits, embedding rows as stored
CONFIGS = {
    "mix": config([mixer(), mixer(left(heads=3, kv_heads=3, dim=8, vdim=8, window=5, dims=8, scaling=None),
                                  right(heads=2, dim=8, vdim=8, decay=[0.9, 1.0]), ls=1.0, rs=-0.5), mixer(left(window=40))],
                  [moe(), None, moe(ff=16, experts=8, top=4, groups=(4, 2), shared=(8, 3.0))]),
    "plain": config([mixer(left(heads=2, kv_heads=1, window=None, dims=0), right(heads=1, dim=40, vdim=8, decay=[1.0])),
                     mixer(left(heads=5, kv_heads=1, dim=12, vdim=10, window=64, dims=4, base=100.0), right(heads=4, dim=5, vdim=7))],
                    [moe(ff=32, experts=3, top=1, groups=None, shared=None, scale=1.0), moe(experts=4, top=3, groups=(4, 3))],
                    width=48, vocab=131, softcap=None, scale=None),
    "one": config([mixer(left(heads=1, kv_heads=1, dim=32, vdim=16, scale=0.4, window=1), right(heads=2, dim=20, vdim=8, decay=[0.5, 0.0])),
                   mixer(left(heads=1, kv_heads=1, dim=20, vdim=40, window=29, dims=20, scaling={"factor": 2.0, "low": 0.5, "high": 8.0, "original": 30}),
                         right(heads=1, dim=33, vdim=1, decay=[0.99]))],
                  [moe(ff=8, experts=1, top=1, groups=(1, 1), shared=(8, 1.0)), moe(ff=9, experts=10, top=4, groups=(2, 1))],
                  width=42, vocab=97, softcap=3.0, eps=1e-6, scale=6.5),
    # (shapes of a kind the tensor-core kernels take in bfloat16: keys of 64 and 128 with values as wide or twice as wide)
    "wide": config([mixer(left(heads=6, kv_heads=2, dim=64, vdim=64, window=37, dims=64), right(heads=2, dim=64, vdim=96)),
                    mixer(left(heads=2, kv_heads=1, dim=128, vdim=128, window=75, dims=32), right(heads=3, dim=128, vdim=64)),
                    mixer(left(heads=4, kv_heads=4, dim=32, vdim=64, window=200, dims=16), right(heads=1, dim=32, vdim=128), ls=0.4)],
                   [moe(ff=40, experts=12, top=3, groups=(3, 2)), moe(ff=32, experts=9, top=2, groups=(3, 1), shared=(64, 2.0)), None],
                   width=96, vocab=257),
    "two": config([mixer(left(heads=2, kv_heads=1, dim=8, vdim=8, dims=4), right(heads=2, dim=8, vdim=8)) for _ in range(2)],
                  [moe(ff=48), moe(ff=48)], width=56, vocab=89, softcap=30.0),
}


def draw(name: str, need, rng) -> np.ndarray:
    """One tensor's values. Matrices N(0, 1/fan_in) so activations stay of order one; norm gains 1 + N(0, 0.2); sink
    scores of a score's size; router rows wide enough that few choices are close calls and no score is at 0 or 1."""
    shape = tuple(need.shape)
    if name.endswith(".sink"):
        return rng.normal(0.0, 1.5, shape)
    if need.init == "ones":
        return 1.0 + rng.normal(0.0, 0.2, shape)
    if name == "embed":  # (the head too: small enough that a token's own row does not decide the next token)
        return rng.normal(0.0, 0.15, shape)
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
    bfloat16, cached per request (the interface `compare` takes)."""

    def __init__(self, cfg: dict, weights: dict):
        self.cfg, self.w = cfg, plain_weights(weights)
        self._cache = {}

    def logits(self, rid: str, tokens: list) -> np.ndarray:
        if rid not in self._cache:
            self._cache[rid] = plain_nudorax.forward(self.cfg, self.w, tokens)
        return self._cache[rid]

    def rounded(self, rid: str, tokens: list) -> np.ndarray:
        key = ("rounded", rid)
        if key not in self._cache:
            plain_nudorax.ROUND = bf16_round
            try:
                self._cache[key] = plain_nudorax.forward(self.cfg, self.w, tokens)
            finally:
                plain_nudorax.ROUND = None
        return self._cache[key]

    def tolerance(self, dtype: str, requests: dict) -> float:
        """What a replay may differ by, relative to a row's largest logit. 32-bit: a fixed small number. bfloat16: six
        times what rounding alone does to these very requests' median row (a routed layer takes another expert here
        and there once its input is rounded, and such a row says nothing about rounding), at least 3e-2."""
        if dtype == "float32":
            return 1e-4
        errs = []
        for rid, tokens in requests.items():
            exact = self.logits(rid, tokens)
            errs.append(np.abs(self.rounded(rid, tokens) - exact).max(axis=1) / np.abs(exact).max(axis=1))
        return max(3e-2, 6.0 * float(np.median(np.concatenate(errs))))
