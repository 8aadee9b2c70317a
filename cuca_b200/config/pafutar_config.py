"""Typed configuration of the Pafutar decoder, read from its config.json.

The file is nested: `layers` is a list with one entry per layer (`type` names the mixer, `mixer` holds the mixer's sizes
and constants, `mlp` the feed-forward's or null, and `weights_of`: j says that the layer has no tensors of its own and runs
with layer j's), `embedding.scale`, `max_positions`, `norm.eps`, `postln_alpha`, `vocab`, `width`. Every size and constant
comes from there. A key the file does not have switches its feature off where that makes sense (no `embedding`: rows as
stored; no `mask`: every earlier key is seen; no `mask.keep_first`: the window alone; no `kv_heads`: one key head per query
head; no `vdim`: `dim`; no `scale`: 1/sqrt(dim); `mlp` null: no feed-forward) and is an error otherwise.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Optional

from .bananex_config import _get
from .dupenex_config import _positive
from .model_config import ConfigError

MIXER_TYPES = ("attention",)


@dataclass(frozen=True)
class KeyValueAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: Optional[int]
    keep_first: int

    @staticmethod
    def from_json(m, where):
        heads, dim, mask = _get(m, "heads", int, where), _get(m, "dim", int, where), m.get("mask")
        c = KeyValueAttentionConfig(
            heads=heads, kv_heads=int(m["kv_heads"]) if m.get("kv_heads") is not None else heads, dim=dim,
            scale=float(m["scale"]) if m.get("scale") is not None else dim ** -0.5,
            window=_get(mask, "size", int, where + ".mask") if mask else None,
            keep_first=int(mask.get("keep_first") or 0) if mask else 0)
        _positive(where, heads=c.heads, kv_heads=c.kv_heads, dim=c.dim)
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json `{where}`: {c.kv_heads} kv_heads do not divide {c.heads} heads")
        if m.get("vdim") is not None and int(m["vdim"]) != dim:
            raise ConfigError(f"config.json `{where}.vdim` = {m['vdim']}: the values are the keys, so it must be dim = {dim}")
        if c.window is not None and c.window < 1:
            raise ConfigError(f"config.json `{where}.mask.size` must be at least 1")
        if c.keep_first < 0:
            raise ConfigError(f"config.json `{where}.mask.keep_first` must not be negative")
        return c


@dataclass(frozen=True)
class MlpConfig:
    ff: int

    @staticmethod
    def from_json(m, where):
        kind = str(m.get("kind", "dense"))
        if kind != "dense":
            raise ConfigError(f"config.json `{where}.kind` = `{kind}`; this engine knows: dense")
        c = MlpConfig(_get(m, "ff", int, where))
        _positive(where, ff=c.ff)
        return c


@dataclass(frozen=True)
class PafutarLayer:
    type: str
    mixer: KeyValueAttentionConfig
    mlp: Optional[MlpConfig]
    weights_of: Optional[int]  # the layer whose tensors this one runs with (None: its own)


@dataclass(frozen=True)
class PafutarConfig:
    vocab: int
    width: int
    eps: float
    alpha: float
    embedding_scale: float
    max_positions: int
    layers: tuple

    def weights_layer(self, i: int) -> int:
        """The layer whose tensors layer i runs with: i itself, or where its `weights_of` leads."""
        seen, start = set(), i
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ConfigError(f"config.json `layers[{start}].weights_of` leads back to itself")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    @staticmethod
    def from_json(cfg: dict) -> "PafutarConfig":
        layers = cfg.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json `layers` must be a non-empty list")
        out = []
        for i, entry in enumerate(layers):
            where = f"layers[{i}]"
            kind = _get(entry, "type", str, where)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json `{where}.type` = `{kind}`; this engine knows: {', '.join(MIXER_TYPES)}")
            if not isinstance(entry.get("mixer"), dict):
                raise ConfigError(f"config.json is missing `{where}.mixer`")
            mlp, of = entry.get("mlp"), entry.get("weights_of")
            if of is not None and not (isinstance(of, int) and 0 <= of < len(layers) and of != i):
                raise ConfigError(f"config.json `{where}.weights_of` = {of!r} must name another layer")
            out.append(PafutarLayer(kind, KeyValueAttentionConfig.from_json(entry["mixer"], where + ".mixer"),
                                    MlpConfig.from_json(mlp, where + ".mlp") if mlp else None, of))
        c = PafutarConfig(vocab=_get(cfg, "vocab", int, ""), width=_get(cfg, "width", int, ""),
                          eps=_get(cfg.get("norm"), "eps", float, "norm"), alpha=_get(cfg, "postln_alpha", float, ""),
                          embedding_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)),
                          max_positions=_get(cfg, "max_positions", int, ""), layers=tuple(out))
        _positive("", vocab=c.vocab, width=c.width, max_positions=c.max_positions)
        for i, layer in enumerate(c.layers):
            j = c.weights_layer(i)
            if dataclasses.replace(layer, weights_of=None) != c.layers[j]:
                raise ConfigError(f"config.json `layers[{i}]` runs with the tensors of layers[{j}] but its entry differs")
        return c
