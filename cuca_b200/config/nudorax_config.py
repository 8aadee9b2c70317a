"""Typed configuration of the Nudorax decoder, read from its config.json.

The file is nested: `layers` is a list with one entry per layer (`type` names the mixer, `mixer` holds the mixer's
sizes and constants, `mlp` the feed-forward's or null), `embedding.scale`, `logit_softcap`, `norm.eps`, `vocab`,
`width`. Every size and constant comes from there. A key the file does not have switches its feature off where that
makes sense (no `embedding`: rows as stored; no `logit_softcap`: logits as they are; no `mask`: every earlier key is
seen; no `rot`: no rotation; no `rot.scaling`: plain frequencies; no `kv_heads`: one key head per query head; no `vdim`:
values as wide as keys; no `router.groups`: all experts are one group; no `router.scale`: 1; no `shared`: no shared
expert; `mlp` null: no feed-forward) and is an error otherwise.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .bananex_config import _get
from .dupenex_config import _positive
from .model_config import ConfigError

MIXER_TYPES = ("parallel",)
MAX_POSITIONS = 1 << 20  # the file gives no longest sequence: nothing in the model depends on one


@dataclass(frozen=True)
class WaveScaling:
    """Frequency scaling by wavelength: long waves (above original / low) turn `factor` times slower, short ones (below
    original / high) as they are, those between are blended."""

    factor: float
    low: float
    high: float
    original: float

    @staticmethod
    def from_json(m, where):
        c = WaveScaling(*(_get(m, k, float, where) for k in ("factor", "low", "high", "original")))
        if not (c.factor > 0 and c.low > 0 and c.high > 0 and c.original > 0):
            raise ConfigError(f"config.json `{where}`: factor, low, high and original must be positive")
        return c


@dataclass(frozen=True)
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]
    rot_base: float
    rot_dims: int
    scaling: Optional[WaveScaling]

    @staticmethod
    def from_json(m, where):
        if not isinstance(m, dict):
            raise ConfigError(f"config.json is missing `{where}`")
        heads, dim = _get(m, "heads", int, where), _get(m, "dim", int, where)
        rot, mask = m.get("rot"), m.get("mask")
        sc = rot.get("scaling") if rot else None
        c = WindowAttentionConfig(
            heads=heads, kv_heads=int(m["kv_heads"]) if m.get("kv_heads") is not None else heads, dim=dim,
            vdim=int(m["vdim"]) if m.get("vdim") is not None else dim,
            scale=float(m["scale"]) if m.get("scale") is not None else dim ** -0.5,
            window=_get(mask, "size", int, where + ".mask") if mask else None,
            rot_base=_get(rot, "base", float, where + ".rot") if rot else 10000.0,
            rot_dims=_get(rot, "dims", int, where + ".rot") if rot else 0,
            scaling=WaveScaling.from_json(sc, where + ".rot.scaling") if sc else None)
        _positive(where, heads=c.heads, kv_heads=c.kv_heads, dim=c.dim, vdim=c.vdim)
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json `{where}`: {c.kv_heads} kv_heads do not divide {c.heads} heads")
        if c.rot_dims % 2 or not 0 <= c.rot_dims <= c.dim:
            raise ConfigError(f"config.json `{where}.rot.dims` = {c.rot_dims} must be even and at most dim = {c.dim}")
        if not c.rot_base > 0:
            raise ConfigError(f"config.json `{where}.rot.base` must be positive")
        if c.window is not None and c.window < 1:
            raise ConfigError(f"config.json `{where}.mask.size` must be at least 1")
        return c


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple

    @staticmethod
    def from_json(m, where):
        if not isinstance(m, dict):
            raise ConfigError(f"config.json is missing `{where}`")
        dim, decay = _get(m, "dim", int, where), m.get("decay")
        if not isinstance(decay, list):
            raise ConfigError(f"config.json is missing the list `{where}.decay`")
        c = LightningConfig(heads=_get(m, "heads", int, where), dim=dim,
                            vdim=int(m["vdim"]) if m.get("vdim") is not None else dim,
                            decay=tuple(float(v) for v in decay))
        _positive(where, heads=c.heads, dim=c.dim, vdim=c.vdim)
        if len(c.decay) != c.heads:
            raise ConfigError(f"config.json `{where}.decay` has {len(c.decay)} entries for {c.heads} heads")
        return c


@dataclass(frozen=True)
class ParallelConfig:
    left: WindowAttentionConfig
    right: LightningConfig
    left_scale: float
    right_scale: float

    @staticmethod
    def from_json(m, where):
        return ParallelConfig(WindowAttentionConfig.from_json(m.get("left"), where + ".left"),
                              LightningConfig.from_json(m.get("right"), where + ".right"),
                              _get(m, "left_scale", float, where), _get(m, "right_scale", float, where))


@dataclass(frozen=True)
class ExpertConfig:
    ff: int
    limit: float

    @staticmethod
    def from_json(m, where):
        c = ExpertConfig(_get(m, "ff", int, where), _get(m, "limit", float, where))
        _positive(where, ff=c.ff)
        if not c.limit > 0:
            raise ConfigError(f"config.json `{where}.limit` must be positive")
        return c


@dataclass(frozen=True)
class MlpConfig:
    expert: ExpertConfig
    experts: int
    top: int
    scale: float
    groups: int  # equal runs of neighbouring experts
    keep: int  # how many of them a token may choose from
    shared: Optional[ExpertConfig]

    @staticmethod
    def from_json(m, where):
        kind = str(m.get("kind", "moe"))
        if kind != "moe":
            raise ConfigError(f"config.json `{where}.kind` = `{kind}`; this engine knows: moe")
        r = m.get("router")
        at = where + ".router"
        g = (r.get("groups") or {"count": 1, "keep": 1}) if isinstance(r, dict) else None
        c = MlpConfig(ExpertConfig.from_json(m.get("expert"), where + ".expert"), experts=_get(r, "experts", int, at),
                      top=_get(r, "top", int, at), scale=float(r["scale"]) if r.get("scale") is not None else 1.0,
                      groups=_get(g, "count", int, at + ".groups"), keep=_get(g, "keep", int, at + ".groups"),
                      shared=ExpertConfig.from_json(m["shared"], where + ".shared") if m.get("shared") else None)
        if c.experts < 1 or c.groups < 1 or c.experts % c.groups:
            raise ConfigError(f"config.json `{at}`: {c.groups} groups do not divide {c.experts} experts")
        if not 1 <= c.keep <= c.groups:
            raise ConfigError(f"config.json `{at}.groups.keep` = {c.keep} must lie in 1..{c.groups}")
        if not 1 <= c.top <= c.keep * (c.experts // c.groups):
            raise ConfigError(f"config.json `{at}`: top = {c.top} must lie in 1..{c.keep * (c.experts // c.groups)}, the "
                              "experts of the kept groups")
        return c


@dataclass(frozen=True)
class NudoraxLayer:
    type: str
    mixer: ParallelConfig
    mlp: Optional[MlpConfig]


@dataclass(frozen=True)
class NudoraxConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_softcap: Optional[float]
    layers: tuple

    @staticmethod
    def from_json(cfg: dict) -> "NudoraxConfig":
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
            mlp = entry.get("mlp")
            out.append(NudoraxLayer(kind, ParallelConfig.from_json(entry["mixer"], where + ".mixer"),
                                    MlpConfig.from_json(mlp, where + ".mlp") if mlp else None))
        emb, cap = cfg.get("embedding") or {}, cfg.get("logit_softcap")
        c = NudoraxConfig(vocab=_get(cfg, "vocab", int, ""), width=_get(cfg, "width", int, ""),
                          eps=_get(cfg.get("norm"), "eps", float, "norm"),
                          embedding_scale=float(emb.get("scale", 1.0)), logit_softcap=float(cap) if cap else None,
                          layers=tuple(out))
        if c.vocab < 1 or c.width < 1:
            raise ConfigError("config.json `vocab` and `width` must be positive")
        if c.logit_softcap is not None and c.logit_softcap <= 0:
            raise ConfigError("config.json `logit_softcap` must be positive")
        return c
