"""The Pafutar decoder as a `ModelSpec`.

The stream starts as the embedding row times a constant plus a learned vector of the position. Layers are `sum_norm_shift`
blocks: the sublayers read the stream as it is, the mixer every token mixed with the one before it, and the sum is normed,
x <- N1(alpha x + s1 * mixer(shift(x))), then x <- N2(alpha x + s2 * ff(x)), with a factor per channel on each sublayer's
output. Mixer: the `attention` part without rotation and without a value projection (the values are the keys as projected),
with biases on q and k, an RMS norm per head without a weight, a stored factor on every head's scores, a distance bias with
the slopes 2^(-8 (a + 1) / H) of head a of H, a sliding window beside which the first keys stay visible, and an output gate
per value. Feed-forward: `dense_act` with the square of relu, without biases. A layer entry with `weights_of`: j runs layer
j's parts with a cache and state of its own.
Tensor names: `embed`, `pos`, `head`, `final.norm` and per layer i `l<i>.norm1`, `l<i>.norm2`, `l<i>.ls1`, `l<i>.ls2`,
`l<i>.shift`, `l<i>.mix.*`, `l<i>.mlp.*`.
"""
from __future__ import annotations

from ..config.pafutar_config import PafutarConfig
from ..config.registry import register_architecture
from ..parts.base import PartSpec
from .spec import LayerSpec, ModelSpec, Run


def distance_slopes(heads: int) -> list:
    """The geometric sequence 2^(-8/H), 2^(-16/H), ..., 2^-8 of H heads."""
    return [2.0 ** (-8.0 * (a + 1) / heads) for a in range(heads)]


def _mixer_spec(m, E: int, eps: float, p: str) -> PartSpec:
    return PartSpec("attention",
                    {"width": E, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "values": "keys",
                     "scale": m.scale, "window": m.window, "keep_first": m.keep_first, "position": None, "qk_norm": "unit",
                     "eps": eps, "q_scale": True, "slopes": distance_slopes(m.heads), "gate": True},
                    {"q": p + "q", "k": p + "k", "q_bias": p + "q.b", "k_bias": p + "k.b", "q_scale": p + "temp",
                     "g": p + "g", "o": p + "o"})


def pafutar_spec(cfg: PafutarConfig) -> ModelSpec:
    E, eps = cfg.width, cfg.eps

    def norm(name):
        return PartSpec("rmsnorm", {"width": E, "eps": eps}, {"weight": name})

    layers, at = [], {}  # the layers that have tensors of their own, and where each sits in that list
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is not None:
            continue
        p, has_ff = f"l{i}.", layer.mlp is not None
        at[i] = len(layers)
        names = {"mix": p + "shift", "mixer_scale": p + "ls1"}
        if has_ff:
            names["ffn_scale"] = p + "ls2"
        layers.append(LayerSpec(
            block=PartSpec("sum_norm_shift", {"width": E, "alpha": cfg.alpha}, names),
            mixer=_mixer_spec(layer.mixer, E, eps, p + "mix."), mixer_norm=norm(p + "norm1"),
            feed_forward=PartSpec("dense_act", {"width": E, "inner": layer.mlp.ff, "act": "relu2", "bias": False},
                                  {"up": p + "mlp.up", "down": p + "mlp.down"}) if has_ff else None,
            ffn_norm=norm(p + "norm2") if has_ff else None))
    # every entry of the file is one run with a cache and state of its own
    schedule = [Run(layer=at[cfg.weights_layer(i)], cache=i, owns=True) for i in range(len(cfg.layers))]
    no_ff = {f"l{i}.{name}" for i, layer in enumerate(cfg.layers) if layer.mlp is None for name in ("norm2", "ls2")}
    return ModelSpec(
        architecture="Pafutar", vocab_size=cfg.vocab, width=E, max_positions=cfg.max_positions,
        embedding=PartSpec("embedding", {"vocab": cfg.vocab, "width": E, "scale": cfg.embedding_scale,
                                         "positions": cfg.max_positions}, {"weight": "embed", "positions": "pos"}),
        layers=layers, schedule=schedule, final_norm=norm("final.norm"),
        head=PartSpec("head", {"vocab": cfg.vocab, "width": E}, {"weight": "head"}),
        # a layer without feed-forward has no use for what stands around one, should a file carry it
        ignorable_tensor=lambda name: name in no_ff)


@register_architecture("Pafutar")
def build_pafutar(config_json: dict) -> ModelSpec:
    return pafutar_spec(PafutarConfig.from_json(config_json))
