"""The Nudorax decoder as a `ModelSpec`.

The stream starts as the embedding row times a constant. Layers are `post_norm` blocks: the sublayers read the stream as
it is and only their outputs are normed, x += N1(mixer(x)), then x += N2(ff(x)), with layer norms (weight, no bias).
Every mixer is the `parallel` part without norms of its own, left_scale * left(x) + right_scale * right(x): on the left
sliding-window `attention` (an RMS norm over the whole q and the whole k projection, rotary pairs (i, i + n/2) with
frequencies scaled by wavelength, a stored sink score per head), on the right the `lightning` part (linear attention with
a fixed decay per head behind silu). Feed-forward: `routed_grouped` (sigmoid scores, a choice restricted to the best
groups of experts, capped gated units, a shared expert behind a gate of its own). The head is the embedding table; the
logits pass a smooth cap c tanh(. / c).
Tensor names: `embed`, `final.norm` and per layer i `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.left.*`, `l<i>.mix.right.*`,
`l<i>.mlp.*`.
"""
from __future__ import annotations

from ..config.nudorax_config import MAX_POSITIONS, NudoraxConfig
from ..config.registry import register_architecture
from ..parts.base import PartSpec
from .spec import LayerSpec, ModelSpec, default_schedule

GATE_SLOPE = 1.702  # of the capped unit's sigmoid


def _mixer_spec(m, E: int, eps: float, p: str) -> PartSpec:
    a, r, lp, rp = m.left, m.right, p + "left.", p + "right."
    position = None
    if a.rot_dims:
        scaling = None
        if a.scaling is not None:
            s = a.scaling
            scaling = {"kind": "llama3", "factor": s.factor, "low_freq_factor": s.low, "high_freq_factor": s.high,
                       "original_max_position_embeddings": s.original}
        position = PartSpec("rope", {"head_dim": a.dim, "rotary_dim": a.rot_dims, "theta": a.rot_base, "pairs": "half",
                                     "scaling": scaling})
    left = PartSpec("attention",
                    {"width": E, "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "v_head_dim": a.vdim,
                     "window": a.window, "scale": a.scale, "position": position, "qk_norm": "whole", "eps": eps,
                     "sink": "learned"},
                    {"q": lp + "q", "k": lp + "k", "v": lp + "v", "q_norm": lp + "q.norm", "k_norm": lp + "k.norm",
                     "sink": lp + "sink", "o": lp + "o"})
    right = PartSpec("lightning", {"width": E, "heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay),
                                   "eps": eps},
                     {"q": rp + "q", "k": rp + "k", "v": rp + "v", "g": rp + "g", "norm": rp + "norm", "o": rp + "o"})
    return PartSpec("parallel", {"width": E, "norms": False, "left_scale": m.left_scale, "right_scale": m.right_scale,
                                 "left": left, "right": right})


def _mlp_spec(mlp, E: int, p: str) -> PartSpec:
    names = {"router": p + "router"}
    for e in range(mlp.experts):
        names[f"gate{e}"] = f"{p}e{e}.gate"
        names[f"up{e}"] = f"{p}e{e}.up"
        names[f"down{e}"] = f"{p}e{e}.down"
    params = {"width": E, "inner": mlp.expert.ff, "limit": mlp.expert.limit, "alpha": GATE_SLOPE, "experts": mlp.experts,
              "top": mlp.top, "groups": mlp.groups, "keep": mlp.keep, "scale": mlp.scale}
    if mlp.shared is not None:
        params.update(shared=mlp.shared.ff, shared_limit=mlp.shared.limit)
        names.update({"shared_gate": p + "shared.gate", "shared_up": p + "shared.up", "shared_down": p + "shared.down",
                      "shared_weight": p + "shared.sg"})
    return PartSpec("routed_grouped", params, names)


def nudorax_spec(cfg: NudoraxConfig) -> ModelSpec:
    E, eps = cfg.width, cfg.eps

    def norm(name):
        return PartSpec("layernorm", {"width": E, "eps": eps}, {"weight": name})

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        layers.append(LayerSpec(block=PartSpec("post_norm", {"width": E}),
                                mixer=_mixer_spec(layer.mixer, E, eps, p + "mix."), mixer_norm=norm(p + "norm1"),
                                feed_forward=_mlp_spec(layer.mlp, E, p + "mlp.") if layer.mlp is not None else None,
                                ffn_norm=norm(p + "norm2") if layer.mlp is not None else None))
    no_ff = {f"l{i}.norm2" for i, layer in enumerate(cfg.layers) if layer.mlp is None}
    return ModelSpec(
        architecture="Nudorax", vocab_size=cfg.vocab, width=E, max_positions=MAX_POSITIONS,
        embedding=PartSpec("embedding", {"vocab": cfg.vocab, "width": E, "scale": cfg.embedding_scale},
                           {"weight": "embed"}),
        layers=layers, schedule=default_schedule(len(layers)), final_norm=norm("final.norm"),
        head=PartSpec("head", {"vocab": cfg.vocab, "width": E, "softcap": cfg.logit_softcap}, {"weight": "embed"}),
        # a layer without feed-forward has no use for that sublayer's norm, should a file carry one
        ignorable_tensor=lambda name: name in no_ff)


@register_architecture("Nudorax")
def build_nudorax(config_json: dict) -> ModelSpec:
    return nudorax_spec(NudoraxConfig.from_json(config_json))
