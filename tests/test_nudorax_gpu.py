"""Nudorax on the GPU against the plain implementation (`plain_nudorax.py`): every mechanism alone, whole and cut,
then whole models through the replayer in the four work splits, pages and slots used again, long decoding, and greedy
generation through the entry point and its scheduler."""
import numpy as np
import pytest
import torch

import nudorax_util as nu
import plain_nudorax as pn
import replay_util as ru
from test_bananex_gpu import CUTS, _load, _run_cut

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def rt32():
    from cuca_b200.runtime import Runtime
    return Runtime("cuda:0", torch.float32)


def _f32(a, dev):
    return torch.tensor(np.asarray(a), dtype=torch.float32, device=dev)


def _mixer(m, rt, E, eps, side=None):
    """The part of a mixer (or of one of its sides) as the model builder describes it; tensor names start `l0.mix.`."""
    import cuca_b200.models.model  # noqa: F401  (registers the parts)
    from cuca_b200.config.nudorax_config import NudoraxConfig
    from cuca_b200.models.nudorax import _mixer_spec
    from cuca_b200.parts.base import MIXERS
    cfg = NudoraxConfig.from_json(nu.config([m], [None], width=E, eps=eps))
    spec = _mixer_spec(cfg.layers[0].mixer, E, eps, "l0.mix.")
    if side:
        spec = spec.params[side]
    return MIXERS.get(spec.kind)(spec, rt)


def _weights_for(part, seed, rounded=False):
    rs = np.random.default_rng(seed)
    ws = {name: np.asarray(nu.draw(name, need, rs), dtype=np.float32).astype(np.float64)
          for name, need in part.tensors().items()}
    return {k: nu.bf16_round(v) for k, v in ws.items()} if rounded else ws


def _load_as(part, ws, rt):
    needs = part.tensors()
    part.load(lambda n: torch.tensor(ws[n], dtype=torch.float32 if needs[n].keep_fp32 else rt.dtype, device=rt.device))


def _tol(dtype):
    return 3e-5 if dtype == torch.float32 else 3e-2


# ------------------------------------------------------------------------------------------ norms and sums
@pytest.mark.parametrize("E", [1, 3, 40, 61, 320, 2047, 4096, 6000, 20000, 40000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_layer_norm_of_gathered_rows(rt32, E, dtype):
    """Rows with a mean far from 0 (a variance from the mean square minus the squared mean would lose its digits)."""
    from cuca_b200.kernels import ops
    dev, eps = rt32.device, 1e-5
    rs = np.random.default_rng(E)
    x = (rs.normal(0, 1.5, (5, E)) + np.array([0.0, 300.0, -40.0, 5.0, 1.0])[:, None]).astype(np.float32)
    w = rs.normal(1, 0.3, E)
    rows = torch.tensor([3, 1, 1, 4], dtype=torch.int32, device=dev)
    for gather in (rows, None):
        want = pn.layer_norm(x.astype(np.float64), w, eps)
        want = want[[3, 1, 1, 4]] if gather is not None else want
        out = torch.empty(want.shape, dtype=dtype, device=dev)
        ops.layer_norm(_f32(x, dev), _f32(w, dev), out, eps, gather)
        tol = 2e-4 if dtype == torch.float32 else 1e-2
        assert np.abs(out.float().cpu().numpy() - want).max() < tol * max(1.0, np.abs(want).max())
    many = torch.empty(1100, E, dtype=dtype, device=dev)  # (launches of many rows hold several values a thread)
    ops.layer_norm(_f32(np.tile(x, (220, 1)), dev), _f32(w, dev), many, eps)
    assert np.abs(many.float().cpu().numpy()[-5:] - want).max() < tol * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("rows", [1, 7, 33, 600])
@pytest.mark.parametrize("E", [24, 52, 61, 1024, 5000])
@pytest.mark.parametrize("center", [True, False])
def test_a_normed_sum_of_terms_goes_into_the_stream(rt32, rows, E, center):
    """Terms with factors (a negative one and 0 among them), one of them a contraction's unadded K slices; the rounded
    copy is the new stream's."""
    from cuca_b200.kernels import ops
    dev, eps = rt32.device, 1e-5
    rs = np.random.default_rng(E + rows)
    factors = (0.6, -1.1, 0.0, 2.5)
    parts = [rs.normal(0, 1, (rows, E)) + 2.0 for _ in factors]
    slices = rs.normal(0, 1, (6, rows + 2, E))  # (slabs may be padded beyond the rows)
    parts[3] = slices[:, :rows].sum(0)
    data = _f32(slices, dev)[:, :rows]
    terms = [(_f32(p, dev), c) for p, c in zip(parts[:3], factors)] + [(ops.PartialSums(data, 6), factors[3])]
    y = sum(c * p for p, c in zip(parts, factors))
    w, base = rs.normal(1, 0.3, E), rs.normal(0, 3, (rows, E))
    normed = pn.layer_norm(y, w, eps) if center else pn.rms(y, eps) * w
    x, out = _f32(base, dev), torch.empty(rows, E, dtype=torch.bfloat16, device=dev)
    ops.norm_add(x, terms, _f32(w, dev), eps, out, center=center)
    assert np.abs(x.cpu().numpy() - (base + normed)).max() < 3e-5 * np.abs(base + normed).max()
    assert torch.equal(out, x.to(torch.bfloat16))
    ops.add_terms(x, terms, store=False)
    assert np.abs(x.cpu().numpy() - (base + normed + y)).max() < 3e-5 * np.abs(base + normed + y).max()
    ops.add_terms(x, terms, store=True)
    assert np.abs(x.cpu().numpy() - y).max() < 3e-5 * np.abs(y).max()
    ops.round_rows(x, out)
    assert torch.equal(out, x.to(torch.bfloat16))


def test_a_sublayers_output_collects_and_merges_terms():
    """More contributions than a kernel takes terms; contributions of one factor share a tensor; a scaled view writes
    into the same sum; the 32-bit and the serving precision."""
    from cuca_b200.kernels import ops
    from cuca_b200.runtime import Runtime, SublayerOutput
    for dtype in (torch.float32, torch.bfloat16):
        rt = Runtime("cuda:0", dtype)
        dev, rows, E, K = rt.device, 5, 48, 64
        rs = np.random.default_rng(3)
        y, want = SublayerOutput(rt, rows, E), np.zeros((rows, E))
        for i in range(12):
            a, w = nu.bf16_round(rs.normal(size=(rows, K))), nu.bf16_round(rs.normal(size=(E, K)))
            c = (0.5, 1.0, -2.0)[i % 3]
            y.scaled(c).add_linear(torch.tensor(a, dtype=dtype, device=dev), torch.tensor(w, dtype=dtype, device=dev))
            want += c * (a @ w.T)
            assert len(y.terms) <= ops.MAX_TERMS
        t, fresh = y.scaled(3.0).claim()
        add = rs.normal(size=(rows, E))
        if fresh:
            t.copy_(_f32(add, dev))
        else:
            t.add_(_f32(add, dev))
        want += 3.0 * add
        assert np.abs(y.data.cpu().numpy() - want).max() < 1e-4 * np.abs(want).max()
        assert SublayerOutput(rt, rows, E).data.abs().max() == 0  # nothing written: zeros


@pytest.mark.parametrize("n", [1, 20, 63, 512, 4000])
@pytest.mark.parametrize("rows", [3, 700])
def test_row_norm_gate(rt32, n, rows):
    from cuca_b200.kernels import ops
    dev, eps = rt32.device, 1e-6
    rs = np.random.default_rng(n)
    o, w, g = rs.normal(0, 2, (rows, n)), rs.normal(1, 0.2, n), rs.normal(0, 3, (rows, n + 4))
    want = pn.rms(o, eps) * w * pn.sigmoid(g[:, 4:])
    for dtype in (torch.float32, torch.bfloat16):
        out = torch.empty(rows, n, dtype=dtype, device=dev)
        ops.row_norm_gate(_f32(o, dev), _f32(w, dev), _f32(g, dev)[:, 4:], out, eps)
        assert np.abs(out.float().cpu().numpy() - want).max() < (2e-5 if dtype == torch.float32 else 1e-2) * np.abs(want).max()


# ------------------------------------------------------------------------------------------ lightning attention
LIGHTNINGS = [nu.right(), nu.right(heads=1, dim=40, vdim=8, decay=[1.0]), nu.right(heads=2, dim=128, vdim=96),
              nu.right(heads=5, dim=4, vdim=36), nu.right(heads=1, dim=7, vdim=150, decay=[0.25]),
              nu.right(heads=2, dim=64, vdim=64, decay=[0.999, 0.0]), nu.right(heads=2, dim=200, vdim=5, decay=[0.999, 0.5])]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", LIGHTNINGS)
def test_lightning_alone_whole_and_cut(dtype, m):
    """Three requests in slots 1, 3, 0, whole, one token at a time and in cuts down to two tokens; the state carries
    across every cut and starts at zero although the slots held another request's."""
    from cuca_b200.cache.device import CacheView
    from cuca_b200.runtime import Runtime
    rt = Runtime("cuda:0", dtype)
    dev, E, eps = rt.device, 48, 1e-5
    part = _mixer(nu.mixer(r=m), rt, E, eps, "right")
    ws = _weights_for(part, 5, rounded=True)
    _load_as(part, ws, rt)
    rs = np.random.default_rng(6)
    xs = [nu.bf16_round(rs.normal(0, 1.5, (n, E))) for n in (141, 3, 67)]
    want = [pn.lightning(x, ws, "l0.mix.right.", m, eps) for x in xs]
    state = {k: torch.full((4, *v.shape), 7.0, device=dev) for k, v in part.cache_needs().state.items()}
    for cuts in ([CUTS[0]] * 3, [CUTS[1], CUTS[2], CUTS[1]], [CUTS[2], CUTS[1], CUTS[2]], [[64, 64, 1000], [2, 1], [65, 1000]]):
        for t in state.values():
            t.zero_()  # what the engine does when a slot gets a new request
            t[2] = 5.0  # another request's: must stay as it is

        def fwd(h, step):
            out = rt.stream(torch.zeros(h.shape[0], E, device=dev))
            part.forward(h.to(dtype), out, step, CacheView(None, None, None, 16, -1, state, step.slots))
            return out.data
        got = _run_cut(dev, fwd, xs, cuts, [1, 3, 0], E)
        for a, b in zip(got, want):
            assert np.abs(a - b).max() < _tol(dtype) * max(1.0, np.abs(b).max()), cuts
        assert float(state["memory"][2].min()) == float(state["memory"][2].max()) == 5.0
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("H, d, dv, offset", [(2, 64, 64, 0), (3, 128, 128, 0), (1, 16, 8, 0), (2, 40, 200, 8), (2, 7, 13, 0),
                                              (1, 200, 70, 0), (2, 72, 24, 3), (1, 256, 1, 0)])
def test_lightning_in_chunks_keeps_32_bit_precision(rt32, H, d, dv, offset):
    """The chunked kernels against the recurrence token by token on the very same rounded queries, keys and values: what
    is left is 32-bit rounding, although the products run on 16-bit tensor cores. Requests of one token, of exactly one
    chunk, of one more and of several, from states that are not zero; decays from 0 to 1; unaligned rows too."""
    from cuca_b200.kernels import ops
    from test_bananex_gpu import _step
    dev = rt32.device
    rs = np.random.default_rng(d + dv)
    counts, slots = [1, 64, 65, 2, 230, 63], [4, 0, 5, 2, 6, 3]
    decay = [0.0, 1.0, 0.93][:H] if H > 1 else [0.997]
    cols = H * (2 * d + dv)
    raw = torch.tensor(rs.normal(0, 1.5, (sum(counts), cols + 8 + offset)), dtype=torch.bfloat16, device=dev)
    proj = raw[:, offset:]
    state = rs.normal(0, 1, (8, H, dv, d)).astype(np.float32)
    x = proj[:, :cols].double().cpu().numpy()
    x = nu.bf16_round(pn.silu(x))
    q, k, v = x[:, :H * d].reshape(-1, H, d), x[:, H * d:2 * H * d].reshape(-1, H, d), x[:, 2 * H * d:].reshape(-1, H, dv)
    want, after = np.zeros((len(x), H, dv)), state.astype(np.float64).copy()
    row = 0
    for n, slot in zip(counts, slots):
        for a in range(H):
            S = after[slot, a]
            for t in range(row, row + n):
                S = decay[a] * S + np.outer(v[t, a], k[t, a])
                want[t, a] = S @ q[t, a]
            after[slot, a] = S
        row += n
    starts = np.cumsum([0] + counts[:-1])
    step = _step(dev, [(0, n) for n in counts], slots)
    assert step.req_row0.tolist() == starts.tolist()
    st, out = _f32(state, dev), torch.full((len(x), H * dv), float("nan"), device=dev)
    n_chunks = ops.lightning_chunks(step, torch.bfloat16, d)
    assert n_chunks == 1 + 1 + 2 + 1 + 4 + 1
    ops.lightning_chunked(proj, _f32(decay, dev), st, out, step, n_chunks, H, d, dv)
    got, new = out.cpu().numpy().reshape(want.shape), st.cpu().numpy()
    def close(x, y):  # in the mean to 32-bit precision; a silu that falls between two 16-bit numbers may go either way
        d = np.abs(x - y)
        return np.sqrt(np.mean(d * d)) < 1e-4 * np.sqrt(np.mean(y * y)) and d.max() < 1e-3 * np.abs(y).max()
    for a in range(H):  # (every head by its own size: the one that never decays grows)
        assert close(got[:, a], want[:, a]) and close(new[:, a], after[:, a]), a
    assert np.array_equal(new[[1, 7]], state[[1, 7]])  # slots of no request of the step


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, vdim", [(8, 6), (64, 64), (128, 128)])
def test_lightning_remembers_a_far_token_in_the_slow_head_only(dtype, dim, vdim):
    """Two heads, decays 1 and 1/2. Only the first token writes (its key channel reads an input column that is set on it
    alone); four hundred tokens later the head that never decays still returns its value and the fast head has lost it:
    a lost or mixed-up state, or a decay given to the wrong head, shows."""
    from cuca_b200.cache.device import CacheView
    from cuca_b200.runtime import Runtime
    rt = Runtime("cuda:0", dtype)
    dev, E, eps, n = rt.device, 24, 1e-5, 400
    m = nu.right(heads=2, dim=dim, vdim=vdim, decay=[1.0, 0.5])
    part = _mixer(nu.mixer(r=m), rt, E, eps, "right")
    ws = _weights_for(part, 15, rounded=True)
    p = "l0.mix.right."
    ws[p + "k"][:] = 0.0
    ws[p + "k"][0, 0] = ws[p + "k"][dim, 0] = 10.0  # channel 0 of both heads: written where column 0 is set
    ws[p + "q"][0] = ws[p + "q"][dim] = 0.0
    ws[p + "q"][0, 1] = ws[p + "q"][dim, 1] = 5.0  # ... and read where column 1 is set
    _load_as(part, ws, rt)
    rs = np.random.default_rng(16)
    x = rs.normal(0, 1.0, (n, E))
    x[:, 0:2] = 0.0
    x[0, 0] = 1.0
    x[n - 5:, 1] = 1.0
    x = nu.bf16_round(x)
    want = pn.lightning(x, ws, p, m, eps)
    x2 = x.copy()
    x2[0, 2:] = rs.normal(0, 1.0, E - 2)
    assert np.abs(want[-1] - pn.lightning(x2, ws, p, m, eps)[-1]).max() > 0.3 * np.abs(want[-1]).max()
    for cuts in ([1000], [n - 6] + [1] * 10, [3, 2, 200, 2, 1000]):
        state = {"memory": torch.zeros(4, 2, vdim, dim, device=dev)}

        def fwd(h, step):
            out = rt.stream(torch.zeros(h.shape[0], E, device=dev))
            part.forward(h.to(dtype), out, step, CacheView(None, None, None, 16, -1, state, step.slots))
            return out.data
        got = _run_cut(dev, fwd, [x], [cuts], [2], E)[0]
        # (the last rows: before them the queries read next to nothing, and the norm magnifies it)
        assert np.abs(got - want)[n - 5:].max() < (1e-4 if dtype == torch.float32 else 3e-2) * np.abs(want).max(), cuts
        mem = state["memory"][2].cpu().numpy()
        assert np.abs(mem[0]).max() > 1.0 and np.abs(mem[1]).max() < 1e-30  # 2^-399 of what the first token wrote


# ------------------------------------------------------------------------------------------ window attention
ATTENTIONS = [nu.left(), nu.left(heads=3, kv_heads=3, vdim=16, window=None, dims=0), nu.left(heads=1, kv_heads=1, dim=32, vdim=16, scale=0.4, window=1),
              nu.left(heads=6, kv_heads=2, dim=12, vdim=10, scale=1.2, window=33, scaling=None), nu.left(heads=2, kv_heads=1, dim=8, vdim=300, window=40, dims=2),
              nu.left(heads=4, kv_heads=1, dim=64, vdim=64, window=24, dims=64), nu.left(heads=2, kv_heads=2, dim=136, vdim=40, window=9, dims=100)]


def _pools(part, dtype, dev, pages, bs, fill=0.0):
    kv = part.cache_needs().kv
    shape = (pages, kv.n_kv_heads, bs)
    return (torch.full((*shape, kv.head_dim), fill, dtype=dtype, device=dev),
            torch.full((*shape, kv.v_head_dim or kv.head_dim), fill, dtype=dtype, device=dev))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", ATTENTIONS)
def test_window_attention_alone_whole_and_cut(dtype, m):
    """Pages of 8 positions handed out in a scrambled order and holding NaN before they are written; the norm over the
    whole projection, the scaled rotation, the window and the stored sink scores; whole, one by one and in cuts."""
    from cuca_b200.cache.device import CacheView
    from cuca_b200.runtime import Runtime
    rt = Runtime("cuda:0", dtype)
    dev, E, eps, bs = rt.device, 36, 1e-5, 8
    part = _mixer(nu.mixer(m), rt, E, eps, "left")
    assert part.general and part.sink_learned and part.norm_whole and part.window == (m.get("mask") or {}).get("size")
    ws = _weights_for(part, 7, rounded=True)
    _load_as(part, ws, rt)
    part.prepare(128)
    rs = np.random.default_rng(8)
    xs = [nu.bf16_round(rs.normal(0, 1.5, (n, E))) for n in (75, 20)]
    want = [pn.window_attention(x, ws, "l0.mix.left.", m, eps) for x in xs]
    order = rs.permutation(16).tolist()
    for cuts in ([CUTS[0]] * 2, [CUTS[1], CUTS[2]], [CUTS[2], CUTS[1]]):
        kpool, vpool = _pools(part, dtype, dev, 16, bs, fill=float("nan") if dtype == torch.float32 else 0.0)
        tables = torch.full((4, 16), -1, dtype=torch.int32, device=dev)
        tables[2, :10] = torch.tensor(order[:10], dtype=torch.int32)
        tables[0, :3] = torch.tensor(order[10:13], dtype=torch.int32)

        def fwd(h, step):
            out = rt.stream(torch.zeros(h.shape[0], E, device=dev))
            part.forward(h.to(dtype), out, step, CacheView(kpool, vpool, tables, bs, 0, None, step.slots))
            return out.data
        got = _run_cut(dev, fwd, xs, cuts, [2, 0], E)
        for a, b in zip(got, want):
            assert np.abs(a - b).max() < _tol(dtype) * max(1.0, np.abs(b).max()), cuts
    assert int(rt.err.item()) == 0


def _planted(dtype, dim, vdim, n, far, askers, window, target=16.0, sink=None, dims=0):
    """A window-attention part with a planted key: the last dimension of every q head (behind the rotated ones) reads
    input column 0 and of the k head input column 1; only position `far` has column 1 set, the rows `askers` have
    column 0 set. `scale` is chosen so that the planted score is about `target`, far above the others."""
    from cuca_b200.runtime import Runtime
    rt = Runtime("cuda:0", dtype)
    E, eps, H = 40, 1e-5, 2
    # after the norms over the whole projections the planted entries hold about 8 / sqrt(1 + 64 / size) each
    qn, kn = 8.0 / np.sqrt(1.0 + 63.0 / (H * dim)), 8.0 / np.sqrt(1.0 + 63.0 / dim)
    m = nu.left(heads=H, kv_heads=1, dim=dim, vdim=vdim, scale=target / (qn * kn), window=window, dims=dims)
    part = _mixer(nu.mixer(m), rt, E, eps, "left")
    p = "l0.mix.left."
    ws = _weights_for(part, 13, rounded=True)
    for head in range(H):
        at = head * dim + dim - 1
        ws[p + "q"][at] = 0.0
        ws[p + "q"][at, 0] = 8.0
        ws[p + "q.norm"][at] = 1.0
    ws[p + "k"][dim - 1] = 0.0
    ws[p + "k"][dim - 1, 1] = 8.0
    ws[p + "k.norm"][dim - 1] = 1.0
    if sink is not None:
        ws[p + "sink"][:] = sink
    _load_as(part, ws, rt)
    part.prepare(max(128, n + 8))
    rs = np.random.default_rng(14)
    x = rs.normal(0, 1.0, (n, E))
    x[:, 0:2] = 0.0
    x[far, 1] = 1.0
    x[askers, 0] = 1.0
    return rt, part, m, ws, nu.bf16_round(x), E, eps


def _run_planted(rt, part, ws, m, x, E, eps, cuts, dtype, bs=8):
    from cuca_b200.cache.device import CacheView
    dev, n = rt.device, len(x)
    pages = -(-n // bs)
    rs = np.random.default_rng(3)
    kpool, vpool = _pools(part, dtype, dev, pages + 9, bs)
    tables = torch.full((4, pages + 1), -1, dtype=torch.int32, device=dev)
    tables[1, :pages] = torch.tensor(rs.permutation(pages + 9)[:pages].tolist(), dtype=torch.int32)

    def fwd(h, step):
        out = rt.stream(torch.zeros(h.shape[0], E, device=dev))
        part.forward(h.to(dtype), out, step, CacheView(kpool, vpool, tables, bs, 0, None, step.slots))
        return out.data
    return _run_cut(dev, fwd, [x], [cuts], [1], E)[0]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, vdim", [(16, 24), (64, 64), (32, 96), (128, 128), (96, 96), (128, 40)])
@pytest.mark.parametrize("window", [7, 64, 100, 129, 300])
def test_a_planted_key_just_inside_and_just_outside_the_window(dtype, dim, vdim, window):
    """The planted key is seen by the rows up to `window` - 1 behind it and by no later one: those rows ask for it on
    both sides of the edge, in a prompt, decoded one by one, and with a portion cut between them. A window that is one
    token off changes the row at the edge altogether."""
    n, far = window + 14, 4
    edge = far + window - 1  # the last row that sees it
    rt, part, m, ws, x, E, eps = _planted(dtype, dim, vdim, n, far, slice(edge - 3, n), window)
    p = "l0.mix.left."
    want = pn.window_attention(x, ws, p, m, eps)
    for off in (-1, 1):
        wrong = pn.window_attention(x, ws, p, dict(m, mask={"size": window + off}), eps)
        at = edge if off < 0 else edge + 1
        assert np.abs(want - wrong)[at].max() > 0.2 * np.abs(want).max()
    for cuts in ([1000], [edge - 4] + [1] * 30, [5, 2, edge - 7, 2, 2, 1000], [edge + 1, 2, 1000]):
        got = _run_planted(rt, part, ws, m, x, E, eps, cuts, dtype)
        assert np.abs(got - want).max() < _tol(dtype) * np.abs(want).max(), cuts
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, vdim, dims", [(16, 24, 12), (64, 64, 32), (128, 128, 126), (96, 96, 8)])
def test_one_far_key_that_matters(dtype, dim, vdim, dims):
    """No window: position 3 among five hundred keys, over many pages in a scrambled order, takes nearly all the weight
    of the last rows. Whole, decoded one by one and in portions; through the plain kernel and the tensor-core ones."""
    n, far = 500, 3
    rt, part, m, ws, x, E, eps = _planted(dtype, dim, vdim, n, far, slice(n - 12, n), None, dims=dims)
    p = "l0.mix.left."
    want = pn.window_attention(x, ws, p, m, eps)
    x2 = x.copy()
    x2[far, 2:] += 1.0
    assert np.abs(want[-1] - pn.window_attention(x2, ws, p, m, eps)[-1]).max() > 0.2 * np.abs(want[-1]).max()
    for cuts in ([1000], [n - 14] + [1] * 20, [5, 2, 300, 2, 1000]):
        got = _run_planted(rt, part, ws, m, x, E, eps, cuts, dtype)
        assert np.abs(got - want).max() < _tol(dtype) * np.abs(want).max(), cuts
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, vdim", [(16, 24), (64, 64), (128, 128)])
def test_the_sink_counts_once_and_unscaled(dtype, dim, vdim):
    """A planted score of about 7 against a stored sink score of 7 in head 0 (half the weight each) and of 20 in head 1
    (which returns next to nothing), with a window that starts inside the prompt: a sink left out, counted per key
    chunk, scaled like a score or swapped between heads shows."""
    n, window = 180, 90
    rt, part, m, ws, x, E, eps = _planted(dtype, dim, vdim, n, 110, slice(112, n), window, target=7.0)
    p = "l0.mix.left."
    ws[p + "sink"][:] = [7.0, 20.0]
    _load_as(part, ws, rt)
    want = pn.window_attention(x, ws, p, m, eps)
    for other in ([-30.0, 20.0], [7.0 * m["scale"], 20.0 * m["scale"]], [20.0, 7.0]):
        assert np.abs(want - pn.window_attention(x, dict(ws, **{p + "sink": np.array(other)}), p, m, eps)).max() > 0.1 * np.abs(want).max()
    for cuts in ([1000], [115] + [1] * 80, [60, 2, 61, 2, 1000]):
        got = _run_planted(rt, part, ws, m, x, E, eps, cuts, dtype)
        assert np.abs(got - want).max() < _tol(dtype) * np.abs(want).max(), cuts


@pytest.mark.parametrize("splits, cluster", [(1, True), (2, True), (3, True), (4, False), (8, True), (16, False)])
def test_windows_and_sinks_in_every_merge_of_the_split_key_decode(monkeypatch, splits, cluster):
    """Single tokens whose window covers a part of 1,100 keys dealt to 1 to 16 chunks: chunks wholly outside the window,
    the chunk its edge falls into, and every way of merging."""
    from cuca_b200.kernels import ops
    monkeypatch.setenv("CUCA_DECODE_SPLITS", str(splits))
    monkeypatch.setattr(ops, "CLUSTER_MERGE", cluster)
    n, window = 1100, 393
    far = n - 3 - window + 1  # seen by row n - 3, not by row n - 2
    rt, part, m, ws, x, E, eps = _planted(torch.bfloat16, 128, 128, n, far, slice(n - 6, n), window, target=9.0, sink=9.0)
    want = pn.window_attention(x, ws, "l0.mix.left.", m, eps)
    assert np.abs(want[n - 3] - want[n - 2]).max() > 0.2 * np.abs(want).max()
    got = _run_planted(rt, part, ws, m, x, E, eps, [n - 8] + [1] * 8, torch.bfloat16, bs=16)
    assert np.abs(got - want)[n - 8:].max() < 3e-2 * np.abs(want).max()
    assert int(rt.err.item()) == 0


# ------------------------------------------------------------------------------------------ two mixers side by side
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("ls, rs_", [(0.6, 1.3), (1.0, -0.5), (0.0, 2.0), (-1.5, 0.0)])
def test_both_sides_with_their_factors(dtype, ls, rs_):
    """The pair added to an ordinary stream and gathered as a sublayer's output, over few rows (K slices) and many."""
    from cuca_b200.cache.device import CacheView
    from cuca_b200.runtime import Runtime, SublayerOutput
    from test_bananex_gpu import _step
    rt = Runtime("cuda:0", dtype)
    dev, E, eps, bs = rt.device, 40, 1e-5, 8
    m = nu.mixer(ls=ls, rs=rs_)
    part = _mixer(m, rt, E, eps)
    ws = _weights_for(part, 7, rounded=True)
    _load_as(part, ws, rt)
    part.prepare(1024)
    kv, states = part.cache_needs().kv, part.cache_needs().state
    for n in (1, 9, 700):
        rs = np.random.default_rng(n)
        x, base = nu.bf16_round(rs.normal(0, 1.5, (n, E))), rs.normal(0, 1, (n, E))
        want = pn.parallel(x, ws, "l0.mix.", m, eps)
        for gathered in (False, True):
            pages = -(-n // bs)
            kpool = torch.zeros(pages, kv.n_kv_heads, bs, kv.head_dim, dtype=dtype, device=dev)
            vpool = torch.zeros(pages, kv.n_kv_heads, bs, kv.v_head_dim or kv.head_dim, dtype=dtype, device=dev)
            tables = torch.full((2, pages), -1, dtype=torch.int32, device=dev)
            tables[1] = torch.arange(pages - 1, -1, -1, dtype=torch.int32)
            state = {k: torch.zeros(2, *v.shape, device=dev) for k, v in states.items()}
            step = _step(dev, [(0, n)], [1])
            out = SublayerOutput(rt, n, E) if gathered else rt.stream(_f32(base, dev))
            part.forward(torch.tensor(x, dtype=dtype, device=dev), out, step,
                         CacheView(kpool, vpool, tables, bs, 0, state, step.slots))
            got = out.data.cpu().numpy() - (0 if gathered else base)
            assert np.abs(got - want).max() < _tol(dtype) * max(1.0, np.abs(want).max())
    assert int(rt.err.item()) == 0


# ------------------------------------------------------------------------------------------ routed experts
def _grouped(mlp, E, rt):
    from cuca_b200.config.nudorax_config import MlpConfig
    from cuca_b200.models.nudorax import _mlp_spec
    from cuca_b200.parts.mlp import GroupedExperts
    return GroupedExperts(_mlp_spec(MlpConfig.from_json(mlp, "mlp"), E, "l0.mlp."), rt)


MOES = [(nu.moe(), 48), (nu.moe(ff=8, experts=1, top=1, groups=(1, 1)), 40), (nu.moe(ff=16, experts=4, top=4, groups=(2, 2)), 36),
        (nu.moe(ff=40, experts=39, top=3, groups=(13, 2), shared=(24, 3.0)), 64), (nu.moe(ff=9, experts=100, top=32, groups=(2, 1)), 50),
        (nu.moe(ff=12, experts=5, top=2, groups=(5, 3), shared=None), 24), (nu.moe(ff=16, experts=8, top=3, groups=None, scale=0.3), 32),
        (nu.moe(ff=4, experts=1024, top=7, groups=(8, 2), shared=(8, 0.2)), 16)]


@pytest.mark.parametrize("mlp, E", MOES)
def test_grouped_experts_alone(rt32, mlp, E):
    """Few tokens read only the chosen experts, many tokens run all experts with the unchosen ones weighted 0; both
    against the plain implementation, added to a stream and stored into an unwritten one. Where there are groups they
    decide some of the choices."""
    from cuca_b200.runtime import ResidualStream
    dev = rt32.device
    part = _grouped(mlp, E, rt32)
    ws = _weights_for(part, E)
    _load(part, ws, dev)
    rs = np.random.default_rng(E)
    router = mlp["router"]
    for T in (1, 5, part.SPARSE_MAX_TOKENS, part.SPARSE_MAX_TOKENS + 1, 150):
        f = rs.normal(0, 1.5, (T, E))
        want = pn.routed_ff(f, ws, "l0.mlp.", mlp)
        g = router.get("groups") or {"count": 1, "keep": 1}
        if T == 150 and g["keep"] < g["count"] < router["experts"]:
            free = dict(mlp, router={k: v for k, v in router.items() if k != "groups"})
            assert not np.allclose(want, pn.routed_ff(f, ws, "l0.mlp.", free))
        base = rs.normal(0, 1, (T, E))
        x = _f32(base, dev)
        part.forward(_f32(f, dev), x, None)
        assert np.abs(x.cpu().numpy() - (base + want)).max() < 3e-5 * max(1.0, np.abs(want).max())
        y = ResidualStream.unwritten(rt32, T, E)
        part.forward(_f32(f, dev), y, None)
        assert np.abs(y.data.cpu().numpy() - want).max() < 3e-5 * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("mlp, E", [(nu.moe(), 48), (nu.moe(ff=64, experts=33, top=5, groups=(11, 4)), 64), (nu.moe(ff=40, shared=None), 56),
                                    # (sizes in steps of 32: few tokens go through the tensor-core form)
                                    (nu.moe(ff=96, experts=8, groups=(4, 2), shared=(160, 2.0)), 96),
                                    (nu.moe(ff=32, experts=20, top=5, groups=(5, 3), shared=None), 64),
                                    (nu.moe(ff=64, experts=4, top=4, groups=(2, 2), shared=(32, 1.0)), 100 * 32),
                                    (nu.moe(ff=200, experts=8, top=2, groups=(4, 2), shared=(136, 2.0)), 512)])
@pytest.mark.parametrize("fused", [False, True])
def test_grouped_experts_in_bfloat16(monkeypatch, mlp, E, fused):
    """Few tokens and many (the units in a pass of their own and as the contraction's epilogue) in the serving precision, on the tokens whose choice is clear (rounding cannot change it): the last
    chosen score well above the first open one left, the last kept group's sum well above the next one's."""
    from cuca_b200.runtime import Runtime
    rt = Runtime("cuda:0", torch.bfloat16)
    dev = rt.device
    part = _grouped(mlp, E, rt)
    monkeypatch.setattr(type(part), "FUSED_FROM_WIDTH", 0 if fused else 1 << 30)
    ws = _weights_for(part, E, rounded=True)
    _load_as(part, ws, rt)
    r = mlp["router"]
    top, g = r["top"], r["groups"]
    rs = np.random.default_rng(E + 1)
    for T in ((40, 200, 300) if fused else (1, 2, 7, 13, 17, part.SPARSE_MAX_TOKENS, 40, 200)):
        f = nu.bf16_round(rs.normal(0, 1.5, (T, E)))
        want = pn.routed_ff(f, ws, "l0.mlp.", mlp)
        clear = np.zeros(T, dtype=bool)
        for t in range(T):
            s = pn.sigmoid(f[t] @ ws["l0.mlp.router"].T)
            size = len(s) // g["count"]
            sums = np.sort([sum(sorted(s[i * size:(i + 1) * size])[-2:]) for i in range(g["count"])])[::-1]
            chosen = pn.chosen_experts(s, r)
            rest = [s[e] for e in pn.chosen_experts(s, dict(r, top=g["keep"] * size)) if e not in chosen]
            clear[t] = (g["keep"] == g["count"] or sums[g["keep"] - 1] - sums[g["keep"]] > 0.01) and (not rest or s[chosen[-1]] - max(rest) > 0.01)
        assert clear.sum() >= T // 4
        stream = rt.stream(torch.zeros(T, E, device=dev))  # few rows may leave slices pending on it
        part.forward(torch.tensor(f, dtype=torch.bfloat16, device=dev), stream, None)
        if not clear.any():
            continue
        assert np.abs(stream.data.cpu().numpy() - want)[clear].max() < 3e-2 * np.abs(want).max()


def test_rows_of_padding_may_hold_anything(rt32):
    """Rows that hold NaN or infinities (a captured step's padding) choose some experts and leave the others' rows
    alone."""
    from cuca_b200.kernels import ops
    dev, E, T = rt32.device, 12, 9
    rs = np.random.default_rng(1)
    z = rs.normal(0, 1, (T, E + 1)).astype(np.float32)
    clean = torch.tensor(z, device=dev)
    z[2], z[5, 3], z[7] = np.nan, np.nan, np.inf
    bad = torch.tensor(z, device=dev)
    outs = []
    eye = torch.eye(E + 1, device=dev)  # (the form that makes the logits itself: they are the activations' own entries)
    for few, logits in ((False, clean), (False, bad), (True, clean)):
        idx = torch.empty(T, 4, dtype=torch.int32, device=dev)
        wts = torch.empty(T, 4, dtype=torch.float32, device=dev)
        if few:
            ops.moe_router_grouped(logits, eye, E, 3, 2, 3, 2.0, True, idx, wts)
        else:
            ops.moe_route_grouped(logits, E, 3, 2, 3, 2.0, True, idx, wts)
        outs.append((idx.cpu().numpy(), wts.cpu().numpy()))
    assert ((outs[1][0] >= 0) & (outs[1][0] <= E)).all() and (outs[1][0][:, 3] == E).all()
    for t in (0, 1, 3, 4, 6, 8):
        assert (outs[0][0][t] == outs[1][0][t]).all() and (outs[0][1][t] == outs[1][1][t]).all()
    assert (outs[0][0] == outs[2][0]).all() and (outs[0][1] == outs[2][1]).all()
    for t in range(T):  # no expert twice
        assert len(set(outs[1][0][t].tolist())) == 4


# ------------------------------------------------------------------------------------------ whole models
LENGTHS = {"mix": [1, 2, 5, 16, 33, 64, 97, 130], "plain": [3, 17, 48, 100], "one": [1, 18, 35, 77],
           "wide": [1, 15, 33, 38, 76, 140, 230], "two": [2, 40, 90]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(nu.CONFIGS.items()):
        weights = nu.make_weights(cfg, seed=20 + i)
        out[name] = (nu.write_model(tmp_path_factory.mktemp(f"nudorax_{name}"), cfg, weights), cfg,
                     nu.Oracle(cfg, weights))
    return out


def _requests(name, cfg):
    return {f"r{n}": nu.random_tokens(n, cfg["vocab"], seed=300 + n) for n in LENGTHS[name]}


def test_the_stream_after_every_layer(models):
    from cuca_b200.engine.core import EngineCore
    from cuca_b200.engine.step import StepEntry
    for name in nu.CONFIGS:
        folder, cfg, oracle = models[name]
        core = EngineCore.from_folder(folder, dtype="float32", kv_tokens=128, context_length=128, window_pools="full")
        seen = []
        core.model.layer_hook = lambda n, stream: seen.append(stream.data.cpu().numpy().copy())
        toks = nu.random_tokens(29, cfg["vocab"], 4)
        blocks, slot = core.pools.new_seq(), core.slots.alloc()
        core.cache.clear_slot(slot)
        core.pools.reserve(blocks, len(toks))
        core.stepper.step([StepEntry(blocks, slot, toks, [0])])
        want = []
        pn.forward(cfg, oracle.w, toks, want)
        assert len(seen) == len(want) == len(cfg["layers"])
        for a, b in zip(seen, want):
            assert np.abs(a - b).max() < 1e-4 * np.abs(b).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(nu.CONFIGS))
def test_whole_and_decoded_one_by_one(models, name, dtype):
    folder, cfg, oracle = models[name]
    reqs = _requests(name, cfg)
    for steps in (ru.trace_whole(reqs), ru.trace_tail_one_by_one(reqs, tail=48)):
        got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=8)
        nu.compare(steps, got, reqs, oracle, dtype, allow=0.2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(nu.CONFIGS))
def test_portions_down_to_two_tokens(models, name, dtype):
    folder, cfg, oracle = models[name]
    reqs = _requests(name, cfg)
    for sizes in ((5, 2, 17, 3, 2, 32, 7, 2, 64, 11), (2, 2, 3, 1, 1, 8, 9, 40)):
        steps = ru.trace_portions(reqs, sizes=sizes)
        got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=16)
        nu.compare(steps, got, reqs, oracle, dtype, allow=0.2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(nu.CONFIGS))
def test_mixed_batches_reuse_pages_and_slots(models, name, dtype):
    """Eight and more requests through four (and three) slots and a pool sized for the peak (and, for windows, for the
    window): every slot and most pages serve several requests, whose state must start from zero."""
    folder, cfg, oracle = models[name]
    reqs = _requests(name, cfg)
    reqs.update({f"s{n}": nu.random_tokens(n, cfg["vocab"], seed=900 + n) for n in (4, 9, 23, 31, 58)})
    for live, pools in ((4, "full"), (3, "sized")):
        steps = ru.trace_mixed(reqs, max_live=live, seed=7 + live)
        got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=8, window_pools=pools)
        nu.compare(steps, got, reqs, oracle, dtype, allow=0.2)


def test_32_bit_hardly_depends_on_cuts_or_company(models):
    """In 32-bit a position's logits whole, in portions, decoded and beside other requests differ by rounding alone."""
    folder, cfg, _ = models["mix"]
    reqs = {"a": nu.random_tokens(70, cfg["vocab"], 1), "b": nu.random_tokens(33, cfg["vocab"], 2)}
    whole = ru.trace_whole(reqs)
    ref = ru.run_in_process(folder, "float32", whole, ru.peak_tokens(whole))
    want = {rid: ref[i] for i, rid in enumerate(reqs)}
    for steps in (ru.trace_portions(reqs, sizes=(3, 2, 9, 1, 1, 30)), ru.trace_mixed(reqs, max_live=2, seed=3)):
        got = ru.run_in_process(folder, "float32", steps, ru.peak_tokens(steps))
        pos = {rid: 0 for rid in reqs}
        for s in steps:
            row = 0
            for e in s["entries"]:
                for w in e["want"]:
                    r = want[e["id"]][pos[e["id"]] + w]
                    assert np.abs(got[s["step"]][row] - r).max() < 2e-5 * np.abs(r).max(), (s["step"], e["id"])
                    row += 1
                pos[e["id"]] += len(e["tokens"])


def test_long_decoding(models):
    """Three hundred tokens decoded one by one: every window fills and slides over decoded tokens, pages behind it come
    back and are used again, the state grows token by token."""
    folder, cfg, oracle = models["wide"]
    reqs = {"long": nu.random_tokens(330, cfg["vocab"], 5)}
    steps = ru.trace_tail_one_by_one(reqs, tail=300)
    for dtype in ("float32", "bfloat16"):
        got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=8, window_pools="sized")
        nu.compare(steps, got, reqs, oracle, dtype, allow=0.2)


def test_long_prompts(models):
    folder, cfg, oracle = models["mix"]
    reqs = {"p": nu.random_tokens(610, cfg["vocab"], 8), "q": nu.random_tokens(300, cfg["vocab"], 9)}
    for steps in (ru.trace_whole(reqs), ru.trace_portions(reqs, sizes=(7, 300, 2, 280, 1, 64))):
        for dtype in ("bfloat16", "float32"):
            got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=16)
            nu.compare(steps, got, reqs, oracle, dtype, allow=0.2)  # (few wanted places: one token's other expert is 7 %)


def test_trace_run_as_a_program(models):
    folder, cfg, oracle = models["one"]
    reqs = _requests("one", cfg)
    steps = ru.trace_mixed(reqs, max_live=4, seed=1)
    got = ru.run_subprocess(folder, "float32", steps, ru.peak_tokens(steps))
    nu.compare(steps, got, reqs, oracle, "float32")


# ------------------------------------------------------------------------------------------ the entry point
def _plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(pn.forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]


@pytest.mark.parametrize("name", ["mix", "plain"])
def test_greedy_generation_through_the_entry_point(models, name):
    """`LocalModel.generate`: the scheduler admits, cuts prompts into portions, decodes through captured graphs and
    gives slots to later requests; the tokens are the plain implementation's greedy ones."""
    from cuca_b200 import BatchingConfig, LocalModel, LocalModelConfig
    folder, cfg, oracle = models[name]
    prompts = [nu.random_tokens(n, cfg["vocab"], seed=40 + n) for n in (3, 50, 21, 9, 70)]
    model = LocalModel.load(LocalModelConfig(source=str(folder), dtype="float32", context_length=256,
                                             batching=BatchingConfig(max_sequences=2, prefill_chunk=16)))
    outs = model.generate(prompts, max_tokens=12, temperature=0.0)
    for prompt, out in zip(prompts, outs):
        assert out.tokens == _plain_greedy(cfg, oracle.w, prompt, 12)


def test_command_line_sampling_and_the_prefix_cache_refusal(models):
    import subprocess
    import sys
    from pathlib import Path

    from cuca_b200 import BatchingConfig, LocalModel, LocalModelConfig
    from cuca_b200.cache.pages import StatefulCacheError
    folder, cfg, oracle = models["two"]
    root = Path(__file__).resolve().parent.parent
    r = subprocess.run([sys.executable, "-m", "cuca_b200", "--model-dir", str(folder), "--prompt", "5 9 20 31",
                        "--max-tokens", "6", "--temperature", "0", "--dtype", "float32"],
                       capture_output=True, text=True, cwd=root, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(t) for t in r.stdout.split()] == _plain_greedy(cfg, oracle.w, [5, 9, 20, 31], 6)
    model = LocalModel.load(LocalModelConfig(source=str(folder), dtype="bfloat16", context_length=128))
    prompt = nu.random_tokens(20, cfg["vocab"], 77)
    a = model.generate(prompt, max_tokens=16, temperature=1.0, top_k=20, seed=5).tokens
    b = model.generate(prompt, max_tokens=16, temperature=1.0, top_k=20, seed=5).tokens
    c = model.generate(prompt, max_tokens=16, temperature=1.0, top_k=20, seed=6).tokens
    assert a == b and a != c and all(0 <= t < cfg["vocab"] for t in a)
    with pytest.raises(StatefulCacheError):
        LocalModel.load(LocalModelConfig(source=str(folder), dtype="bfloat16", context_length=128,
                                         batching=BatchingConfig(prefix_cache=True)))


def test_bfloat16_generation_through_captured_graphs(models):
    """The serving precision end to end: prompts in portions, decode steps replayed as CUDA graphs. Where two logits
    nearly tie bfloat16 may take the other branch, so every token it takes must be a near-maximum of the plain
    implementation's logits at its place."""
    from cuca_b200 import BatchingConfig, LocalModel, LocalModelConfig
    folder, cfg, oracle = models["two"]
    prompts = [nu.random_tokens(n, cfg["vocab"], seed=60 + n) for n in (5, 70, 33)]
    model = LocalModel.load(LocalModelConfig(source=str(folder), dtype="bfloat16", context_length=256,
                                             batching=BatchingConfig(max_sequences=4, prefill_chunk=32)))
    assert model.backend.use_graphs
    outs = model.generate(prompts, max_tokens=40, temperature=0.0)
    assert model.backend.graph_steps > 0
    off = 0
    for prompt, out in zip(prompts, outs):
        ref = pn.forward(cfg, oracle.w, prompt + out.tokens)
        for i, tok in enumerate(out.tokens):
            row = ref[len(prompt) - 1 + i]
            off += float(row.max() - row[tok]) > 0.06 * float(np.abs(row).max())
    assert off <= 0.05 * sum(len(o.tokens) for o in outs)  # (a router's near-tie may fall the other way)
