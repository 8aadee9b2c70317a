"""Pafutar without a GPU: the configuration reader and its refusals, the run order with layers that borrow another layer's
tensors, caches per run, tensor names, a folder of random weights, page pools that keep a request's first pages, and
properties of the plain implementation itself."""
import copy

import numpy as np
import pytest

import pafutar_util as pu
import plain_pafutar as pp
from cuca_b200.cache.device import plan_groups
from cuca_b200.cache.pages import NO_BLOCK, GroupLayout, KvPools, StateSlots
from cuca_b200.config.model_config import ConfigError
from cuca_b200.config.pafutar_config import PafutarConfig
from cuca_b200.config.registry import architectures, build_spec
from cuca_b200.models.model import Model
from cuca_b200.models.pafutar import distance_slopes
from cuca_b200.weights.loader import WeightsError, check_tensors


def test_registered_and_read():
    assert "Pafutar" in architectures()
    cfg = PafutarConfig.from_json(pu.CONFIGS["mix"])
    assert (cfg.alpha, cfg.eps, cfg.embedding_scale, cfg.max_positions, len(cfg.layers)) == (1.7, 1e-5, 3.0, 700, 6)
    m = cfg.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.scale, m.window, m.keep_first) == (4, 2, 16, 0.5, 13, 3)
    assert [l.weights_of for l in cfg.layers] == [None, None, 0, None, 1, 2]
    assert [cfg.weights_layer(i) for i in range(6)] == [0, 1, 0, 3, 1, 0]
    assert cfg.layers[1].mlp is None and cfg.layers[3].mlp.ff == 24
    plain = PafutarConfig.from_json(pu.CONFIGS["plain"])
    assert plain.embedding_scale == 1.0 and plain.layers[0].mixer.window is None
    assert plain.layers[3].mixer.scale == 12 ** -0.5 and plain.layers[3].mixer.keep_first == 0
    bare = copy.deepcopy(pu.CONFIGS["two"])
    for l in bare["layers"]:
        del l["mixer"]["kv_heads"], l["mixer"]["mask"]["keep_first"]
    c = PafutarConfig.from_json(bare).layers[0].mixer
    assert c.kv_heads == 2 and c.keep_first == 0 and c.window == 13


@pytest.mark.parametrize("path, value", [
    (("layers", 0, "type"), "conv_only"), (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "dim"), 0),
    (("layers", 0, "mixer", "vdim"), 8), (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 0, "mixer", "mask", "size"), None),
    (("layers", 0, "mixer", "mask", "keep_first"), -1), (("layers", 0, "mlp", "kind"), "moe"), (("layers", 0, "mlp", "ff"), 0),
    (("norm",), None), (("postln_alpha",), None), (("max_positions",), None), (("max_positions",), 0), (("layers", 3, "mixer"), None),
    (("layers", 2, "weights_of"), 2), (("layers", 2, "weights_of"), 9), (("layers", 2, "weights_of"), 1), (("layers",), []),
    (("layers", 2, "mixer", "scale"), 0.25), (("layers", 0, "weights_of"), 2)])
def test_refusals(path, value):
    cfg = copy.deepcopy(pu.CONFIGS["mix"])
    node = cfg
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    with pytest.raises(ConfigError):
        PafutarConfig.from_json(cfg)


def test_run_order_caches_and_tensors():
    spec = build_spec(pu.CONFIGS["mix"])
    assert [r.layer for r in spec.runs()] == [0, 1, 0, 2, 1, 0] and [r.cache for r in spec.runs()] == list(range(6))
    assert spec.max_positions == 700
    model = Model(spec)
    needs = model.cache_needs()
    assert len(needs) == 6 and all(n.state["shift"].shape == (60,) and n.state["shift"].dtype == "float32" for n in needs.values())
    # (one row per key and value, and a factor per key)
    assert all(n.kv.v_head_dim == 0 and n.kv.key_scale for n in needs.values())
    assert [(n.kv.window, n.kv.keep_first) for n in needs.values()] == [(13, 3), (5, 1), (13, 3), (40, 9), (5, 1), (13, 3)]
    names = set(model.tensor_needs())
    want = {"embed", "pos", "head", "final.norm"}
    for i in (0, 1, 3):
        want |= {f"l{i}.norm1", f"l{i}.ls1", f"l{i}.shift"} | {f"l{i}.mix.{t}" for t in ("q", "q.b", "k", "k.b", "temp", "g", "o")}
        if i != 1:
            want |= {f"l{i}.norm2", f"l{i}.ls2", f"l{i}.mlp.up", f"l{i}.mlp.down"}
    assert names == want
    shapes = {n: tuple(t.shape) for n, t in model.tensor_needs().items()}
    assert shapes["pos"] == (700, 60) and shapes["l0.mix.g"] == (64, 60) and shapes["l0.mix.k.b"] == (32,) and shapes["l0.mix.temp"] == (4,)
    # what stands around a feed-forward is of no use to a layer without one
    check_tensors(model.tensor_needs(), {**shapes, "l1.norm2": (60,), "l1.ls2": (60,)}, spec.ignorable_tensor, "a folder")
    with pytest.raises(WeightsError):
        check_tensors(model.tensor_needs(), {**shapes, "l2.norm1": (60,)}, spec.ignorable_tensor, "a folder")


def test_layers_with_one_mask_share_a_group_of_pages():
    needs = Model(build_spec(pu.CONFIGS["mix"])).cache_needs()
    groups = plan_groups(needs, kv_tokens=640, block_size=8, max_sequences=2, max_step_tokens=16)
    assert sorted((g.window, g.keep_first, g.cache_ids, g.n_blocks) for g in groups) == [
        (5, 1, (1, 4), 2 * (3 + 2 + 1)), (13, 3, (0, 2, 5), 2 * (4 + 2 + 1)), (40, 9, (3,), 2 * (7 + 2 + 2))]


def test_distance_slopes():
    assert distance_slopes(8) == [0.5, 0.25, 0.125, 0.0625, 0.03125, 0.015625, 0.0078125, 0.00390625]
    assert distance_slopes(1) == [2.0 ** -8] and np.allclose(distance_slopes(3), pp.slopes(3))


# ------------------------------------------------------------------------------------------ pages of the kept first keys
def _pools(window, keep, n=64, bs=4, full=None):
    groups = [GroupLayout(1, 16, window, (0,), n, None, keep)]
    if full:
        groups.append(GroupLayout(1, 16, None, (1,), full))
    return KvPools(groups, bs)


@pytest.mark.parametrize("window, keep", [(6, 0), (6, 1), (6, 4), (6, 5), (1, 3), (9, 30), (40, 2)])
def test_pages_of_the_first_keys_stay(window, keep):
    """At every length exactly the pages that a later query may still see are held, plus those of the step itself."""
    bs = 4
    kv = _pools(window, keep)
    s = kv.new_seq()
    for length in range(1, 90):
        kv.reserve(s, length)
        s.length = length
        kv.release_window(s)
        table = s.tables[0]
        for i, page in enumerate(table):
            seen = any(j < keep or j >= length - (window - 1) for j in range(i * bs, min((i + 1) * bs, length))) or (i + 1) * bs > length
            assert (page != NO_BLOCK) == seen, (length, i)
        kv.check()
    held = [p for p in s.tables[0] if p != NO_BLOCK]
    assert len(held) == len(set(held)) == kv.pools[0].used
    kv.release(s)
    kv.check()
    assert kv.pools[0].free == kv.pools[0].n_blocks


def test_a_cached_prefix_needs_the_kept_pages_and_the_windows():
    kv = _pools(6, 5, n=16, full=32)
    ids = list(range(40))
    a = kv.new_seq()
    kv.reserve(a, 20)
    a.length = 20
    kv.release_window(a)
    assert [p != NO_BLOCK for p in a.tables[0]] == [True, True, False, True, True]
    kv.publish(a, ids[:20])
    b = kv.new_seq_with_prefix(ids[:20] + [77])
    assert b.length == 20 and b.tables[0][2] == NO_BLOCK
    assert b.tables[0][:2] == a.tables[0][:2] and b.tables[0][3:] == a.tables[0][3:]
    kv.check()
    kv.release_window(b)
    kv.release(b)
    kv.check()
    c = kv.new_seq_with_prefix(ids[:13])  # the window there would need page 2, which is gone
    assert c.length == 8
    kv.release(c)
    kv.release(a)
    kv.check()


def test_a_long_prompt_is_admitted_to_pools_sized_for_its_window():
    """A windowed pool holds a window, the kept pages and one step's tokens per request, however long the prompt is."""
    from cuca_b200.engine.scheduler import Request, Scheduler, SchedulerConfig
    from test_scheduler import FakeBackend

    class Backend(FakeBackend):
        def run(self, plans):
            out = super().run(plans)
            for p in plans:
                self.pools.release_window(p.seq.blocks)
            return out

    needs = Model(build_spec(pu.CONFIGS["two"])).cache_needs()
    step = 16
    groups = plan_groups(needs, kv_tokens=4 * 256, block_size=4, max_sequences=2, max_step_tokens=step)
    kv, slots = KvPools(groups, 4), StateSlots(2)
    assert all(g.n_blocks * 4 < 200 for g in groups)
    sched = Scheduler(kv, slots, Backend(kv), SchedulerConfig(2, step, step, 256, ()), seed_source=lambda: 42)
    seqs = [sched.submit(Request(list(range(200)), max_tokens=8)) for _ in range(3)]
    sched.run_until_done()
    assert all(s.finish_reason == "length" and len(s.completion) == 8 for s in seqs)
    kv.check()
    assert all(p.free == p.n_blocks for p in kv.pools)


def test_a_folder_of_random_weights_can_be_described():
    from cuca_b200.weights.loader import RandomSource
    needs = Model(build_spec(pu.CONFIGS["one"])).tensor_needs()
    src = RandomSource(needs, 3, 0.02)
    assert src.shapes()["l1.mix.q"] == (20, 42)


# ------------------------------------------------------------------------------------------ the plain implementation
def test_plain_visible_and_shift():
    assert pp.visible(9, {"size": 3, "keep_first": 2}).tolist() == [0, 1, 7, 8, 9]
    assert pp.visible(3, {"size": 3, "keep_first": 2}).tolist() == [0, 1, 2, 3]
    assert pp.visible(1, {"size": 1, "keep_first": 5}).tolist() == [0, 1]
    assert pp.visible(4, {"size": 2}).tolist() == [3, 4] and pp.visible(2, None).tolist() == [0, 1, 2]
    x = np.array([[1.0, 2.0], [5.0, 6.0]])
    assert np.allclose(pp.shift(x, np.array([0.25, 1.0])), [[0.75, 0.0], [4.0, 2.0]])


def test_plain_attention_of_equal_keys_is_the_distance_softmax():
    """Zero projections with a constant key bias: every score is the same but for the distance, every value is the bias."""
    m = pu.attn(heads=2, kv_heads=1, dim=4, window=3, keep=1, scale=0.7)
    T, E = 7, 5
    w = {"q": np.zeros((8, E)), "q.b": np.ones(8), "k": np.zeros((4, E)), "k.b": np.array([1.0, 2.0, 3.0, 4.0]), "temp": np.array([1.0, -2.0]),
         "g": np.zeros((8, E)), "o": np.eye(8)}
    out = pp.attention(np.zeros((T, E)), w, "", m, 0.0)
    assert np.allclose(out, np.tile([0.5, 1.0, 1.5, 2.0], 2))  # (the weights add up to 1 whatever they are; the gate is 1/2)
    w["k"] = np.zeros((4, E))
    w["k"][0, 0] = 1.0
    h = np.zeros((T, E))
    h[0, 0] = 100.0  # only the kept first key differs
    w["q"], w["q.b"] = np.zeros((8, E)), np.zeros(8)
    out = pp.attention(h, w, "", m, 1e-9)[-1].reshape(2, 4)[:, 0]
    for a, slope in enumerate((2.0 ** -4, 2.0 ** -8)):  # (queries of nothing score 0 everywhere)
        e = np.exp(-slope * np.array([6.0, 2.0, 1.0, 0.0]))
        assert np.isclose(out[a], 0.5 * (1.0 + 100.0 * e[0] / e.sum()), rtol=1e-6)


def test_plain_model_depends_on_what_it_should():
    """Positions, the previous token's share, layer scales and heads' factors all reach the logits."""
    cfg = pu.CONFIGS["one"]
    w = pu.plain_weights(pu.make_weights(cfg, 5))
    toks = pu.random_tokens(12, cfg["vocab"], 1)
    base = pp.forward(cfg, w, toks)
    for name in ("pos", "l0.shift", "l1.ls1", "l1.ls2", "l2.ls1", "l1.mix.temp", "l1.mix.q.b", "l2.mix.k.b", "l1.mix.g", "final.norm"):
        changed = dict(w)
        changed[name] = w[name] * 1.3 + 0.05
        assert np.abs(pp.forward(cfg, changed, toks) - base).max() > 1e-4, name
