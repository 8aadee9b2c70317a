"""Seeded random Pafutar configurations (sizes off the beaten track, every feature on or off) through the replayer: whole,
with the last tokens one by one, in portions and in mixed batches through four slots, against the plain implementation in
both dtypes; and layer by layer in bfloat16."""
import numpy as np
import pytest

import pafutar_util as pu
import plain_pafutar as pp
import replay_util as ru

pytestmark = pytest.mark.gpu


def random_config(seed: int) -> dict:
    rs = np.random.default_rng(6000 + seed)
    pick = lambda xs: xs[int(rs.integers(len(xs)))]  # noqa: E731
    layers = []
    for i in range(int(rs.integers(1, 6))):
        if i and rs.random() < 0.3:  # borrow an earlier layer's tensors (through another borrower, perhaps)
            of = int(rs.integers(i))
            layers.append(dict(layers[of], weights_of=of))
            continue
        heads = pick([1, 2, 3, 4, 6, 8, 12, 16])
        kv = pick([k for k in (1, 2, 3, 4, 6, 8, 12) if heads % k == 0])
        m = pu.attn(heads=heads, kv_heads=kv, dim=pick([8, 16, 16, 24, 32, 40, 48, 64, 64, 80, 96, 128]), scale=pick([None, 0.1, 0.3, 0.7]),
                    window=pick([1, 2, 7, 16, 33, 64, 65, 120, None]), keep=pick([0, 1, 3, 4, 16, 17, 65]))
        layers.append(pu.layer(m, ff=pick([None, 8, 12, 20, 36, 40, 64, 96, 200])))
    return pu.config(layers, width=pick([24, 36, 41, 52, 64, 72, 96, 100, 128, 200, 256]), vocab=int(rs.integers(50, 700)),
                     eps=pick([1e-5, 1e-6, 1e-3]), alpha=pick([1.0, 0.7, 1.4, 2.3, 3.0]), scale=pick([None, 1.0, 4.0, 11.0]), max_positions=256)


@pytest.mark.parametrize("seed", list(range(14)))
def test_random_configuration(tmp_path, seed):
    cfg = random_config(seed)
    weights = pu.make_weights(cfg, seed=100 + seed)
    folder = pu.write_model(tmp_path / "m", cfg, weights)
    oracle = pu.Oracle(cfg, weights)
    reqs = {f"r{n}": pu.random_tokens(n, cfg["vocab"], seed=7 * seed + n) for n in (1, 2, 19, 41, 70, 150)}
    for dtype in ("float32", "bfloat16"):
        tol = oracle.tolerance(dtype, reqs)
        for steps in (ru.trace_whole(reqs), ru.trace_tail_one_by_one(reqs, tail=40),
                      ru.trace_portions(reqs, sizes=(7, 2, 33, 2, 3, 64, 5)), ru.trace_mixed(reqs, max_live=4, seed=seed)):
            got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=16)
            pu.compare(steps, got, reqs, oracle, dtype, tol)


@pytest.mark.parametrize("seed", list(range(14)))
def test_every_layer_on_the_engines_own_input_in_bfloat16(tmp_path, seed):
    """The stream after every layer of a bfloat16 run against the plain layer (rounded inputs) on the stream the engine
    itself had before it: nothing carries over from layer to layer."""
    from cuca_b200.engine.core import EngineCore
    from cuca_b200.engine.step import StepEntry
    cfg = random_config(seed)
    weights = pu.make_weights(cfg, seed=100 + seed)
    w = pu.plain_weights(weights)
    core = EngineCore.from_folder(pu.write_model(tmp_path / "m", cfg, weights), dtype="bfloat16", kv_tokens=256,
                                  context_length=256, window_pools="full")
    toks, seen = pu.random_tokens(150, cfg["vocab"], seed), []
    core.model.layer_hook = lambda i, s: seen.append(s.data.double().cpu().numpy().copy())
    blocks, slot = core.pools.new_seq(), core.slots.alloc()
    core.cache.clear_slot(slot)
    core.pools.reserve(blocks, len(toks))
    core.stepper.step([StepEntry(blocks, slot, toks, [0])])
    x = pp.embed(cfg, w, toks)
    pp.ROUND = pu.bf16_round
    try:
        for i, layer in enumerate(cfg["layers"]):
            j = i
            while cfg["layers"][j].get("weights_of") is not None:
                j = cfg["layers"][j]["weights_of"]
            y = pp.run_layer(x, w, f"l{j}.", layer, cfg["postln_alpha"], cfg["norm"]["eps"])
            err = np.abs(y - seen[i]).max(axis=1) / np.abs(y).max(axis=1)
            assert np.median(err) < 8e-3 and err.max() < 3e-2, (seed, i)
            x = seen[i]
    finally:
        pp.ROUND = None
