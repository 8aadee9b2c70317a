"""Seeded random Nudorax configurations (sizes off the beaten track, every feature on or off) through the replayer:
whole, with the last tokens one by one, in portions and in mixed batches through four slots, against the plain
implementation in both dtypes; and layer by layer in bfloat16."""
import numpy as np
import pytest

import nudorax_util as nu
import plain_nudorax as pn
import replay_util as ru

pytestmark = pytest.mark.gpu


def random_config(seed: int) -> dict:
    rs = np.random.default_rng(4000 + seed)
    pick = lambda xs: xs[int(rs.integers(len(xs)))]  # noqa: E731
    width = pick([24, 36, 41, 52, 64, 72, 96, 100, 128, 200, 256])
    mixers, mlps = [], []
    for _ in range(int(rs.integers(1, 5))):
        heads = pick([1, 2, 4, 6, 8, 12])
        kv = pick([k for k in (1, 2, 3, 4, 6, 8, 12) if heads % k == 0])
        dim = pick([8, 16, 24, 32, 48, 64, 80, 96, 128])
        dims = pick([0, 2, dim // 4 * 2, dim, dim])
        scaling = pick([None, {"factor": pick([2.0, 4.0, 32.0]), "low": pick([0.5, 1.0]), "high": pick([2.0, 4.0, 9.0]),
                               "original": pick([16, 64, 500, 8192])}])
        l = nu.left(heads=heads, kv_heads=kv, dim=dim, vdim=pick([dim // 2, dim, dim, 2 * dim, dim + 8, 16, 48, 64]),
                    scale=pick([None, 0.3, 2.0 * dim ** -0.5]), window=pick([1, 2, 7, 16, 33, 64, 65, 120, None]),
                    base=pick([100.0, 10000.0, 500000.0]), dims=dims, scaling=scaling if dims else None)
        rh = pick([1, 2, 3, 4, 6, 8])
        r = nu.right(heads=rh, dim=pick([4, 8, 16, 24, 32, 64, 96, 128]), vdim=pick([8, 16, 20, 32, 48, 64, 128, 160]),
                     decay=[float(1.0 - 2.0 ** -rs.integers(1, 12)) for _ in range(rh)])
        mixers.append(nu.mixer(l, r, ls=pick([0.3, 0.8, 1.0, 1.4]), rs=pick([0.5, 1.0, 1.2, -0.7])))
        if rs.random() < 0.15:
            mlps.append(None)
            continue
        experts = pick([1, 2, 3, 4, 8, 12, 16, 33])
        groups = pick([None] + [g for g in (1, 2, 3, 4, 6, 8, 11) if experts % g == 0])
        open_ = experts
        if groups:
            keep = int(rs.integers(1, groups + 1))
            open_ = keep * (experts // groups)
        mlps.append(nu.moe(ff=pick([8, 12, 16, 20, 24, 40, 64, 96]), limit=pick([0.7, 2.0, 7.0]), experts=experts,
                           top=int(rs.integers(1, min(open_, 6) + 1)), groups=(groups, keep) if groups else None,
                           scale=pick([1.0, 0.4, 2.5]), shared=pick([None, (8, 1.0), (40, 3.0), (24, 0.5)])))
    return nu.config(mixers, mlps, width=width, vocab=int(rs.integers(50, 700)), eps=pick([1e-5, 1e-6]),
                     softcap=pick([None, 5.0, 30.0, 50.0]), scale=pick([None, 1.0, 3.0, float(np.sqrt(width))]))


@pytest.mark.parametrize("seed", list(range(12)))
def test_random_configuration(tmp_path, seed):
    cfg = random_config(seed)
    weights = nu.make_weights(cfg, seed=100 + seed)
    folder = nu.write_model(tmp_path / "m", cfg, weights)
    oracle = nu.Oracle(cfg, weights)
    reqs = {f"r{n}": nu.random_tokens(n, cfg["vocab"], seed=7 * seed + n) for n in (1, 2, 19, 41, 70, 150)}
    for dtype in ("float32", "bfloat16"):
        for steps in (ru.trace_whole(reqs), ru.trace_tail_one_by_one(reqs, tail=40),
                      ru.trace_portions(reqs, sizes=(7, 2, 33, 2, 3, 64, 5)),
                      ru.trace_mixed(reqs, max_live=4, seed=seed)):
            got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=16)
            # bfloat16: a token whose scores nearly tie may go to another expert, and what it then leaves in keys and
            # states moves the tokens behind it; the test below takes every sublayer by itself
            nu.compare(steps, got, reqs, oracle, dtype, allow=0.3, tol32=3e-4)


def _choice_gap(scores, router):
    """How far a token's choice is from another one: the last chosen score above the best open one that was left, the
    last kept group's sum above the first dropped one's."""
    g = router.get("groups") or {"count": 1, "keep": 1}
    size = len(scores) // g["count"]
    chosen = pn.chosen_experts(scores, router)
    rest = [scores[e] for e in pn.chosen_experts(scores, dict(router, top=g["keep"] * size)) if e not in chosen]
    gap = scores[chosen[-1]] - max(rest) if rest else 1.0
    if g["keep"] < g["count"]:
        sums = np.sort([sum(sorted(scores[i * size:(i + 1) * size])[-2:]) for i in range(g["count"])])[::-1]
        gap = min(gap, sums[g["keep"] - 1] - sums[g["keep"]])
    return gap


@pytest.mark.parametrize("seed", list(range(12)))
def test_every_layer_on_the_engines_own_input_in_bfloat16(tmp_path, seed):
    """The stream after every layer of a bfloat16 run against the plain layer (rounded inputs) on the stream the engine
    itself had before it: nothing carries over from layer to layer, so every token whose choice of experts is clear must
    agree closely, and those whose choice is not are few."""
    from cuca_b200.engine.core import EngineCore
    from cuca_b200.engine.step import StepEntry
    cfg = random_config(seed)
    weights = nu.make_weights(cfg, seed=100 + seed)
    w, eps = nu.plain_weights(weights), cfg["norm"]["eps"]
    core = EngineCore.from_folder(nu.write_model(tmp_path / "m", cfg, weights), dtype="bfloat16", kv_tokens=256,
                                  context_length=256, window_pools="full")
    toks, seen = nu.random_tokens(150, cfg["vocab"], seed), []
    core.model.layer_hook = lambda i, s: seen.append(s.data.double().cpu().numpy().copy())
    blocks, slot = core.pools.new_seq(), core.slots.alloc()
    core.cache.clear_slot(slot)
    core.pools.reserve(blocks, len(toks))
    core.stepper.step([StepEntry(blocks, slot, toks, [0])])
    x = w["embed"][np.asarray(toks)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    pn.ROUND = nu.bf16_round
    try:
        for i, layer in enumerate(cfg["layers"]):
            y = x + pn.layer_norm(pn.parallel(x, w, f"l{i}.mix.", layer["mixer"], eps), w[f"l{i}.norm1"], eps)
            clear = np.ones(len(toks), dtype=bool)
            if layer.get("mlp"):
                scores = pn.sigmoid(nu.bf16_round(y) @ w[f"l{i}.mlp.router"].T)
                clear = np.array([_choice_gap(s, layer["mlp"]["router"]) > 0.01 for s in scores])
                f = pn.routed_ff(y, w, f"l{i}.mlp.", layer["mlp"])
                # (an output that nearly vanishes, one expert of a score near 0 for instance, is magnified by its norm)
                clear &= f.std(axis=1) > 0.2 * np.median(f.std(axis=1))
                y = y + pn.layer_norm(f, w[f"l{i}.norm2"], eps)
            err = np.abs(y - seen[i]).max(axis=1) / np.abs(y).max(axis=1)
            assert np.median(err) < 8e-3 and err[clear].max() < 4e-2 and (err > 4e-2).mean() < 0.04, (seed, i)
            assert clear.mean() > 0.5
            x = seen[i]
    finally:
        pn.ROUND = None
