"""Nudorax without a GPU: the configuration reader and its refusals, caches per layer, tensor names, a folder of random
weights, the rotation tables, and properties of the plain implementation itself."""
import copy
import math

import numpy as np
import pytest

import nudorax_util as nu
import plain_nudorax as pn
from cuca_b200.config.model_config import ConfigError
from cuca_b200.config.nudorax_config import NudoraxConfig
from cuca_b200.config.registry import architectures, build_spec
from cuca_b200.models.model import Model
from cuca_b200.weights.loader import WeightsError, check_tensors


def test_registered_and_read():
    assert "Nudorax" in architectures()
    cfg = NudoraxConfig.from_json(nu.CONFIGS["mix"])
    assert cfg.logit_softcap == 12.0 and cfg.eps == 1e-5 and cfg.embedding_scale == 1.6 and len(cfg.layers) == 3
    m = cfg.layers[0].mixer
    assert (m.left_scale, m.right_scale) == (0.75, 1.25)
    a, r = m.left, m.right
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.rot_dims, a.rot_base) == (4, 2, 16, 24, 13, 12, 5000.0)
    assert (a.scaling.factor, a.scaling.low, a.scaling.high, a.scaling.original) == (6.0, 1.0, 4.0, 60.0)
    assert (r.heads, r.dim, r.vdim, r.decay) == (3, 12, 20, (0.5, 0.9375, 1.0 - 2.0 ** -7))
    f = cfg.layers[0].mlp
    assert (f.expert.ff, f.expert.limit, f.experts, f.top, f.groups, f.keep, f.scale) == (24, 1.5, 6, 2, 3, 2, 1.75)
    assert (f.shared.ff, f.shared.limit) == (40, 0.8) and cfg.layers[1].mlp is None
    plain = NudoraxConfig.from_json(nu.CONFIGS["plain"])
    assert plain.logit_softcap is None and plain.embedding_scale == 1.0
    assert plain.layers[0].mixer.left.window is None and plain.layers[0].mixer.left.rot_dims == 0
    assert plain.layers[0].mlp.shared is None and (plain.layers[0].mlp.groups, plain.layers[0].mlp.keep) == (1, 1)
    # absent keys: as many key heads as heads, values as wide as keys, scale 1
    bare = copy.deepcopy(nu.CONFIGS["mix"])
    left, rightside = bare["layers"][0]["mixer"]["left"], bare["layers"][0]["mixer"]["right"]
    del left["kv_heads"], left["vdim"], rightside["vdim"], bare["layers"][0]["mlp"]["router"]["scale"]
    c = NudoraxConfig.from_json(bare).layers[0]
    assert c.mixer.left.kv_heads == 4 and c.mixer.left.vdim == 16 and c.mixer.right.vdim == 12 and c.mlp.scale == 1.0


@pytest.mark.parametrize("path, value", [
    (("layers", 0, "type"), "attention"), (("layers", 0, "mixer"), None), (("layers", 0, "mixer", "left"), None),
    (("layers", 0, "mixer", "right"), None), (("layers", 0, "mixer", "left_scale"), None),
    (("layers", 0, "mixer", "left", "kv_heads"), 3), (("layers", 0, "mixer", "left", "dim"), 0),
    (("layers", 0, "mixer", "left", "rot", "dims"), 7), (("layers", 0, "mixer", "left", "rot", "dims"), 18),
    (("layers", 0, "mixer", "left", "mask", "size"), 0), (("layers", 0, "mixer", "left", "rot", "scaling", "factor"), 0.0),
    (("layers", 0, "mixer", "left", "rot", "scaling", "original"), None),
    (("layers", 0, "mixer", "right", "decay"), [0.5, 0.9]), (("layers", 0, "mixer", "right", "decay"), None),
    (("layers", 0, "mlp", "router", "top"), 5), (("layers", 0, "mlp", "router", "groups", "count"), 4),
    (("layers", 0, "mlp", "router", "groups", "keep"), 4), (("layers", 0, "mlp", "kind"), "dense"),
    (("layers", 0, "mlp", "expert", "limit"), 0.0), (("layers", 0, "mlp", "shared", "ff"), 0),
    (("layers", 0, "mlp", "expert"), None), (("norm",), None), (("logit_softcap",), -2.0), (("vocab",), None)])
def test_refusals_name_the_key(path, value):
    cfg = copy.deepcopy(nu.CONFIGS["mix"])
    node = cfg
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        NudoraxConfig.from_json(cfg)
    assert str(path[-1]) in str(e.value) or str(path[-2]) in str(e.value)


def test_every_layer_keeps_a_window_and_a_state():
    for cfg in nu.CONFIGS.values():
        spec = build_spec(cfg)
        assert [r.layer for r in spec.runs()] == [r.cache for r in spec.runs()] == list(range(len(cfg["layers"])))
        needs = Model(spec, runtime=None).cache_needs()
        for i, layer in enumerate(cfg["layers"]):
            a, r = layer["mixer"]["left"], layer["mixer"]["right"]
            kv = needs[i].kv
            assert (kv.n_kv_heads, kv.head_dim, kv.v_head_dim or kv.head_dim) == (a["kv_heads"], a["dim"], a["vdim"])
            assert kv.window == (a["mask"]["size"] if a.get("mask") else None)
            assert {k: v.shape for k, v in needs[i].state.items()} == {"right.memory": (r["heads"], r["vdim"], r["dim"])}


def test_tensor_names_and_shapes():
    cfg = nu.CONFIGS["mix"]
    model = Model(build_spec(cfg), runtime=None)
    needs = model.tensor_needs()
    shapes = {n: tuple(t.shape) for n, t in needs.items()}
    want = {"embed": (199, 60), "final.norm": (60,), "l0.norm1": (60,), "l0.norm2": (60,), "l0.mix.left.q": (64, 60),
            "l0.mix.left.k": (32, 60), "l0.mix.left.v": (48, 60), "l0.mix.left.q.norm": (64,), "l0.mix.left.k.norm": (32,),
            "l0.mix.left.sink": (4,), "l0.mix.left.o": (60, 96), "l0.mix.right.q": (36, 60), "l0.mix.right.k": (36, 60),
            "l0.mix.right.v": (60, 60), "l0.mix.right.g": (60, 60), "l0.mix.right.norm": (60,), "l0.mix.right.o": (60, 60),
            "l0.mlp.router": (6, 60), "l0.mlp.e5.gate": (24, 60), "l0.mlp.e5.up": (24, 60), "l0.mlp.e5.down": (60, 24),
            "l0.mlp.shared.gate": (40, 60), "l0.mlp.shared.up": (40, 60), "l0.mlp.shared.down": (60, 40),
            "l0.mlp.shared.sg": (1, 60)}
    for name, shape in want.items():
        assert shapes[name] == shape, name
    # no head of its own (the embedding table serves), no norm of a sublayer that is not there
    assert "head" not in shapes and "l1.norm2" not in shapes and "l1.norm1" in shapes and "l0.mlp.e6.up" not in shapes
    check_tensors(needs, shapes, model.spec.ignorable_tensor)
    check_tensors(needs, dict(shapes, **{"l1.norm2": (60,)}), model.spec.ignorable_tensor)
    shapes["l0.mix.left.q.norm"] = (16,)  # over the whole projection, not per head
    with pytest.raises(WeightsError) as e:
        check_tensors(needs, shapes)
    assert [w[0] for w in e.value.wrong_shape] == ["l0.mix.left.q.norm"]


def test_a_folder_of_random_weights(tmp_path):
    from cuca_b200.weights.loader import FolderSource, write_model_folder
    cfg = nu.CONFIGS["two"]
    model = Model(build_spec(cfg), runtime=None)
    write_model_folder(tmp_path, cfg, model.tensor_needs(), seed=3, norm_std=0.2)
    model.check_weights(FolderSource(tmp_path))


@pytest.mark.parametrize("dim, rot", [(16, {"base": 5000.0, "dims": 12, "scaling": nu.WAVES}),
                                      (40, {"base": 250000.0, "dims": 32, "scaling": {"factor": 16.0, "low": 2.0, "high": 5.0, "original": 333.5}}),
                                      (6, {"base": 100.0, "dims": 6, "scaling": {"factor": 1.0, "low": 1.0, "high": 4.0, "original": 64}}),
                                      (20, {"base": 500.0, "dims": 20})])
def test_rotation_tables_are_the_plain_frequencies(dim, rot):
    """The engine's cos and sin tables, as the model builder asks for them, against angles made from the plain
    implementation's frequencies."""
    from cuca_b200.models.nudorax import _mixer_spec
    from cuca_b200.parts.rope import RotaryEncoding
    m = nu.mixer(nu.left(dim=dim, base=rot["base"], dims=rot["dims"], scaling=rot.get("scaling")))
    layer = NudoraxConfig.from_json(nu.config([m], [None])).layers[0]
    part = RotaryEncoding(_mixer_spec(layer.mixer, 60, 1e-5, "l0.mix.").params["left"].params["position"], None)
    assert part.pairs == "half" and part.rotary_dim == rot["dims"]
    cos, sin = part.host_tables(400)
    f = pn.frequencies(rot)
    ang = np.arange(400)[:, None] * f[None, :]
    assert np.abs(cos.numpy() - np.cos(ang)).max() < 3e-5 and np.abs(sin.numpy() - np.sin(ang)).max() < 3e-5
    plain = np.array([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)])
    sc = rot.get("scaling")
    if sc and sc["factor"] > 1:  # short waves as they are, long ones slowed down, something in between
        assert f[0] == plain[0] and f[-1] == pytest.approx(plain[-1] / sc["factor"])
        ratio = f / plain
        assert (np.diff(ratio) <= 1e-12).all() and ((ratio < 0.999) & (ratio > 1.001 / sc["factor"])).any()
    else:
        assert np.allclose(f, plain)


# ------------------------------------------------------------------------------------------ the plain implementation
@pytest.mark.parametrize("name", list(nu.CONFIGS))
def test_plain_is_causal_and_carries_the_first_token(name):
    cfg = nu.CONFIGS[name]
    w = nu.plain_weights(nu.make_weights(cfg, 1))
    toks = nu.random_tokens(30, cfg["vocab"], 2)
    a = pn.forward(cfg, w, toks)
    b = pn.forward(cfg, w, toks[:20] + nu.random_tokens(10, cfg["vocab"], 3))
    assert np.array_equal(a[:20], b[:20]) and not np.allclose(a[20:], b[20:])
    c = pn.forward(cfg, w, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
    assert not np.allclose(a[-1], c[-1])
    if cfg.get("logit_softcap"):
        assert np.abs(a).max() < cfg["logit_softcap"]


def _attention_weights(E, d, dv, H, seed):
    rs = np.random.default_rng(seed)
    return rs, {"q": rs.normal(size=(H * d, E)), "k": rs.normal(size=(d, E)), "v": rs.normal(size=(dv, E)),
                "q.norm": rs.normal(1, 0.2, H * d), "k.norm": rs.normal(1, 0.2, d), "sink": rs.normal(size=H),
                "o": np.eye(H * dv)}


def test_plain_window_attention_with_few_keys():
    """A window of two: the third token sees itself and the second, and a head's weights leave room for exp(sink)."""
    E, d, dv = 6, 4, 3
    rs, w = _attention_weights(E, d, dv, 2, 1)
    h = rs.normal(size=(3, E))
    m = {"heads": 2, "kv_heads": 1, "dim": d, "vdim": dv, "scale": 0.6, "mask": {"size": 2}}
    out = pn.window_attention(h, w, "", m, 1e-6)
    q = pn.rms(w["q"] @ h[2], 1e-6) * w["q.norm"]  # over both heads at once
    k = [pn.rms(w["k"] @ h[j], 1e-6) * w["k.norm"] for j in range(3)]
    v = [w["v"] @ h[j] for j in range(3)]
    for a in range(2):
        e = [math.exp(0.6 * float(q[a * d:(a + 1) * d] @ k[j])) for j in range(3)]
        den = e[1] + e[2] + math.exp(w["sink"][a])
        assert np.allclose(out[2, a * dv:(a + 1) * dv], (e[1] * v[1] + e[2] * v[2]) / den)
    wider = pn.window_attention(h, w, "", dict(m, mask={"size": 3}), 1e-6)
    assert np.allclose(wider[:2], out[:2]) and not np.allclose(wider[2], out[2])
    assert np.allclose(wider, pn.window_attention(h, w, "", {k_: v_ for k_, v_ in m.items() if k_ != "mask"}, 1e-6))


def test_plain_rotation_turns_scores_by_the_distance():
    """Turned queries and keys score by their distance alone, and the part of a head behind `dims` is left alone."""
    rs = np.random.default_rng(2)
    rot = {"base": 30.0, "dims": 4, "scaling": {"factor": 3.0, "low": 0.5, "high": 2.0, "original": 12}}
    v = np.tile(rs.normal(size=(1, 1, 6)), (9, 1, 1))
    t = pn.rotate_half(v, rot)
    assert np.array_equal(t[:, :, 4:], v[:, :, 4:]) and np.array_equal(t[0], v[0])
    s = t[:, 0] @ t[:, 0].T
    for gap in range(1, 6):
        assert np.allclose(np.diagonal(s, gap), s[0, gap])


def test_plain_lightning_is_a_decaying_sum():
    """o_t = sum_j decay^(t - j) (q_t . k_j) v_j with silu on all three, then one norm over the concatenated heads."""
    E, d, dv, T = 5, 4, 3, 7
    rs = np.random.default_rng(3)
    w = {"q": rs.normal(size=(2 * d, E)), "k": rs.normal(size=(2 * d, E)), "v": rs.normal(size=(2 * dv, E)),
         "g": rs.normal(size=(2 * dv, E)), "norm": rs.normal(1, 0.2, 2 * dv), "o": np.eye(2 * dv)}
    h = rs.normal(size=(T, E))
    decay = [0.8, 1.0]
    got = pn.lightning(h, w, "", {"heads": 2, "dim": d, "vdim": dv, "decay": decay}, 1e-6)
    q, k, v = (pn.silu(h @ w[n].T) for n in ("q", "k", "v"))
    for t in range(T):
        o = np.concatenate([sum(decay[a] ** (t - j) * (q[t, a * d:(a + 1) * d] @ k[j, a * d:(a + 1) * d])
                                * v[j, a * dv:(a + 1) * dv] for j in range(t + 1)) for a in range(2)])
        assert np.allclose(got[t], o / np.sqrt(np.mean(o * o) + 1e-6) * w["norm"] * pn.sigmoid(w["g"] @ h[t]))


def test_plain_layer_norm_takes_the_mean_off():
    v = np.array([[1.0, 3.0, 5.0], [100.0, 100.0, 103.0]])
    got = pn.layer_norm(v, np.array([1.0, 2.0, 1.0]), 0.0)
    assert np.allclose(got[0], [-2 / math.sqrt(8 / 3), 0.0, 2 / math.sqrt(8 / 3)])
    assert np.allclose(got[1], [-1 / math.sqrt(2), -2 / math.sqrt(2), 2 / math.sqrt(2)])


def test_plain_experts_are_chosen_within_the_best_groups():
    router = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    s = np.array([0.9, 0.1, 0.6, 0.5, 0.2, 0.7])  # group sums 1.0, 1.1, 0.9: the best expert sits in a lesser group
    assert pn.chosen_experts(s, router) == [2, 3]
    router["groups"]["keep"] = 2
    assert pn.chosen_experts(s, router) == [0, 2]
    router["groups"]["keep"] = 3
    assert pn.chosen_experts(s, router) == [0, 5] == pn.chosen_experts(s, {"experts": 6, "top": 2})
    big = {"experts": 6, "top": 1, "groups": {"count": 2, "keep": 1}}  # only the two largest of a group count
    assert pn.chosen_experts(np.array([0.5, 0.5, 0.5, 0.0, 0.9, 0.3]), big) == [4]
    ones = {"experts": 3, "top": 1, "groups": {"count": 3, "keep": 1}}  # groups of one
    assert pn.chosen_experts(np.array([0.2, 0.4, 0.3]), ones) == [1]


def test_plain_routed_weights_and_the_shared_expert():
    mlp = nu.moe(ff=4, limit=0.7, experts=4, top=2, groups=None, scale=2.0, shared=(3, 0.4))
    rs = np.random.default_rng(5)
    E = 6
    w = {"router": rs.normal(size=(4, E)), "shared.sg": rs.normal(size=(1, E))}
    for name, n in [(f"e{e}.", 4) for e in range(4)] + [("shared.", 3)]:
        w[name + "gate"], w[name + "up"], w[name + "down"] = rs.normal(size=(n, E)), rs.normal(size=(n, E)), rs.normal(size=(E, n))
    f = rs.normal(size=(3, E))
    got = pn.routed_ff(f, w, "", mlp)

    def unit(p, x, limit):
        g, u = np.minimum(w[p + "gate"] @ x, limit), np.clip(w[p + "up"] @ x, -limit, limit)
        return w[p + "down"] @ (g / (1 + np.exp(-1.702 * g)) * (u + 1))
    for t in range(3):
        s = 1 / (1 + np.exp(-(w["router"] @ f[t])))
        a, b = sorted(range(4), key=lambda e: -s[e])[:2]
        want = 2.0 * (s[a] * unit(f"e{a}.", f[t], 0.7) + s[b] * unit(f"e{b}.", f[t], 0.7))
        want = want + unit("shared.", f[t], 0.4) / (1 + math.exp(-float(w["shared.sg"][0] @ f[t])))
        assert np.allclose(got[t], want)
