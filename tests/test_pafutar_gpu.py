"""Pafutar on the GPU against the plain implementation (`plain_pafutar.py`): every mechanism alone, whole and cut, then
whole models through the replayer in the four work splits, pages and slots used again, long decoding, and greedy generation
through the entry point and its scheduler."""
import numpy as np
import pytest
import torch

import pafutar_util as pu
import plain_pafutar as pp
import replay_util as ru
from test_bananex_gpu import CUTS, _run_cut, _step

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def rt32():
    from cuca_b200.runtime import Runtime
    return Runtime("cuda:0", torch.float32)


def _rt(dtype):
    from cuca_b200.runtime import Runtime
    return Runtime("cuda:0", dtype)


def _t(a, dev, dtype=torch.float32):
    return torch.tensor(np.asarray(a), dtype=dtype, device=dev)


def _tol(dtype):
    return 3e-5 if dtype == torch.float32 else 2.5e-2


# ------------------------------------------------------------------------------------------ embedding and stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E", [1, 30, 36, 64, 2060])
def test_embedding_with_learned_positions(dtype, E):
    from cuca_b200.kernels import ops
    rt = _rt(dtype)
    rs = np.random.default_rng(E)
    table, pos = pu.bf16_round(rs.normal(0, 1, (17, E))), pu.bf16_round(rs.normal(0, 1, (50, E)))
    toks, ps = [3, 16, 0, 3, 9], [49, 0, 7, 7, 21]
    out = torch.empty(5, E, device=rt.device)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=rt.device)  # noqa: E731
    ops.embed_pos(_t(table, rt.device, dtype), _t(pos, rt.device, dtype), i32(toks), i32(ps), out, rt.err, 2.7)
    assert np.abs(out.cpu().numpy() - (table[toks] * 2.7 + pos[ps])).max() < 1e-5 and int(rt.err.item()) == 0
    # a position without a row is reported, not read
    ops.embed_pos(_t(table, rt.device, dtype), _t(pos, rt.device, dtype), i32([1]), i32([50]), out[:1], rt.err, 1.0)
    assert np.abs(out[0].cpu().numpy() - table[1]).max() < 1e-6 and int(rt.err.item()) == 1


@pytest.mark.parametrize("rows", [1, 5, 300])
@pytest.mark.parametrize("E", [7, 52, 61, 1024, 5000, 9000, 40000])
def test_norm_of_the_sum(rt32, rows, E):
    """Terms with factors, one of them a contraction's unadded K slices, times a factor per channel, on top of alpha x; the
    rounded copy is the new stream's. The last width is more than a block holds."""
    from cuca_b200.kernels import ops
    if E > 5000 and rows > 5:
        pytest.skip("one size of many rows is enough")
    dev, eps, alpha = rt32.device, 1e-5, 1.6
    rs = np.random.default_rng(E + rows)
    slices = rs.normal(0, 1, (6, rows + 2, E))  # (slabs may be padded beyond the rows)
    part = rs.normal(0, 1, (rows, E))
    terms = [(_t(part, dev), 0.7), (ops.PartialSums(_t(slices, dev)[:, :rows], 6), 1.0)]
    y, s, w, base = 0.7 * part + slices[:, :rows].sum(0), rs.normal(1, 0.3, E), rs.normal(1, 0.3, E), rs.normal(0, 3, (rows, E))
    for scale in (s, None):
        want = pp.sum_norm(base, y, alpha, 1.0 if scale is None else scale, w, eps)
        x, out = _t(base, dev), torch.empty(rows, E, dtype=torch.bfloat16, device=dev)
        ops.sum_norm(x, terms, None if scale is None else _t(scale, dev), _t(w, dev), alpha, eps, out)
        assert np.abs(x.cpu().numpy() - want).max() < 2e-5 * np.abs(want).max()
        assert torch.equal(out, x.to(torch.bfloat16))


@pytest.mark.parametrize("E", [5, 52, 61, 1024, 4100, 8192])
@pytest.mark.parametrize("fused", [True, False])
def test_token_shift_with_and_without_the_norm_before_it(rt32, E, fused):
    """Three requests in slots 2, 3, 0, whole (so that several blocks of rows share a request), one by one and in cuts: the
    row before the first comes from the slot, the last row stays there, other slots are left alone."""
    from cuca_b200.kernels import ops
    dev, eps, alpha = rt32.device, 1e-5, 0.9
    rs = np.random.default_rng(E)
    lengths = (290, 9, 37) if E < 4000 else (23, 9, 5)
    w, s, mix = rs.normal(1, 0.3, E), rs.normal(1, 0.3, E), rs.uniform(0, 1, E)
    xs = [rs.normal(0, 2, (n, E)) for n in lengths]
    ys = [rs.normal(0, 1, (n, E)) for n in lengths]
    new = [pp.sum_norm(x, y, alpha, s, w, eps) if fused else x for x, y in zip(xs, ys)]
    want = [np.hstack([pp.shift(x, mix), x]) for x in new]
    both = [np.hstack([x, y]) for x, y in zip(xs, ys)]
    for cuts in ([CUTS[0]] * 3, [CUTS[1], CUTS[2], CUTS[1]], [[281, 4, 1000], [2, 7], [1000]]):
        kept = torch.zeros(5, E, device=dev)
        kept[1], kept[4] = 7.0, -3.0

        def fwd(h, step):
            x, y = h[:, :E].contiguous(), h[:, E:].contiguous()
            out, x_out = torch.empty_like(x), torch.full_like(x, float("nan"))
            if fused:
                ops.sum_norm_shift(x, [(y, 1.0)], _t(s, dev), _t(w, dev), alpha, eps, x_out, _t(mix, dev), kept, out, step)
            else:
                ops.shift_rows(x, _t(mix, dev), kept, out, step)
                x_out = x
            return torch.cat([out, x_out], dim=1)
        got = _run_cut(dev, fwd, both, cuts, [2, 3, 0], E)
        for a, b in zip(got, want):
            assert np.abs(a - b).max() < 2e-5 * np.abs(b).max(), cuts
        assert bool((kept[1] == 7.0).all()) and bool((kept[4] == -3.0).all())
        for slot, x in zip((2, 3, 0), new):
            assert np.abs(kept[slot].cpu().numpy() - x[-1]).max() < 1e-5 * np.abs(x).max()


def test_shift_skips_padding_rows(rt32):
    """Rows of slot -1 (a captured step's padding) leave every slot alone and become zeros, beside rows that are real."""
    from cuca_b200.engine.step import StepBatch
    from cuca_b200.kernels import ops
    dev, E = rt32.device, 24
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)  # noqa: E731
    step = StepBatch.single_tokens(i32([0] * 4), i32([5, 9, 0, 0]), i32([1, 0, -1, -1]), i32([0, 1, 2, 3]), 16)
    rs = np.random.default_rng(0)
    x, kept0, mix = rs.normal(0, 1, (4, E)), rs.normal(0, 1, (3, E)), rs.uniform(0, 1, E)
    for fused in (True, False):
        kept, out, x_out = _t(kept0, dev), torch.full((4, E), 9.0, device=dev), torch.full((4, E), 9.0, device=dev)
        one = torch.ones(E, device=dev)
        if fused:
            ops.sum_norm_shift(_t(x, dev), [(torch.zeros(4, E, device=dev), 1.0)], None, one, 1.0, 1e-5, x_out, _t(mix, dev), kept, out, step)
            new = pp.rms(x, 1e-5)
        else:
            ops.shift_rows(_t(x, dev), _t(mix, dev), kept, out, step)
            new = x
        for row, slot in ((0, 1), (1, 0)):
            assert np.abs(out[row].cpu().numpy() - (new[row] + (kept0[slot] - new[row]) * mix)).max() < 1e-5
            assert np.abs(kept[slot].cpu().numpy() - new[row]).max() < 1e-5
        assert np.abs(kept[2].cpu().numpy() - kept0[2]).max() < 1e-6 and not out[2:].any()


@pytest.mark.parametrize("E", [24, 64])
def test_a_deferred_sum_reads_the_same_through_every_reader(rt32, E):
    """A layer's last sum is left to the next reader: the stream's data, its rounded copy, a norm, and the next layer's
    shift all see it; dropping it leaves nothing behind."""
    from cuca_b200.parts.base import PartSpec
    from cuca_b200.parts.norm import RMSNorm
    from cuca_b200.runtime import ResidualStream, SublayerOutput
    for dtype in DTYPES:
        rt = _rt(dtype)
        dev, eps, n = rt.device, 1e-5, 6
        rs = np.random.default_rng(E)
        base, y, w, s, mix = rs.normal(0, 2, (n, E)), rs.normal(0, 1, (n, E)), rs.normal(1, 0.2, E), rs.normal(1, 0.2, E), rs.uniform(0, 1, E)
        norm = RMSNorm(PartSpec("rmsnorm", {"width": E, "eps": eps}, {"weight": "w"}), rt)
        norm.load(lambda name: _t(w, dev))
        want = pp.sum_norm(base, y, 1.3, s, w, eps)

        def deferred():
            stream = ResidualStream(rt, _t(base, dev))
            out = SublayerOutput(rt, n, E)
            t, fresh = out.claim()
            assert fresh
            t.copy_(_t(y, dev))
            stream.defer_sum_norm(out, norm, 1.3, _t(s, dev))
            return stream
        tol = 1e-5 if dtype == torch.float32 else 1e-2
        step = _step(dev, [(0, n)], [1])
        assert np.abs(deferred().data.cpu().numpy() - want).max() < 2e-5
        assert np.abs(deferred().rounded().float().cpu().numpy() - want).max() < tol * np.abs(want).max()
        assert np.abs(deferred().take()[0].cpu().numpy() - want).max() < 2e-5
        assert np.abs(norm.forward(deferred()).float().cpu().numpy() - pp.rms(want, eps) * w).max() < 2 * tol * np.abs(want).max()
        stream = deferred()
        h = stream.shifted(_t(mix, dev), torch.zeros(2, E, device=dev), step)
        assert np.abs(h.float().cpu().numpy() - pp.shift(want, mix)).max() < tol * np.abs(want).max()
        assert np.abs(stream.data.cpu().numpy() - want).max() < 2e-5
        stream = deferred()
        stream.add(torch.ones(n, E, device=dev))
        assert np.abs(stream.data.cpu().numpy() - want - 1).max() < 2e-5
        stream = deferred()
        stream.drop_pending()
        assert stream._unsummed is None


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, inner", [(48, 40), (64, 96), (30, 7), (256, 1024), (72, 300)])
@pytest.mark.parametrize("bias", [False, True])
def test_squared_relu_unit(dtype, width, inner, bias):
    """The activation as the contraction's epilogue (every form: few rows, column pieces, whole tiles) and as a pass."""
    from cuca_b200.parts.base import PartSpec
    from cuca_b200.parts.mlp import DenseActivation
    rt = _rt(dtype)
    names = {"up": "p.up", "down": "p.down"} | ({"up_bias": "p.up.b", "down_bias": "p.down.b"} if bias else {})
    part = DenseActivation(PartSpec("dense_act", {"width": width, "inner": inner, "act": "relu2", "bias": bias}, names), rt)
    rs = np.random.default_rng(inner)
    ws = {n: pu.bf16_round(rs.normal(0, 1, need.shape) / np.sqrt(need.shape[-1])) for n, need in part.tensors().items()}
    part.load(lambda n: _t(ws[n], rt.device, dtype))
    for T in (1, 9, 100, 257, 600):
        f = pu.bf16_round(rs.normal(0, 1.5, (T, width)))
        u = np.maximum(f @ ws["p.up"].T + (ws["p.up.b"] if bias else 0), 0)
        want = (u * u) @ ws["p.down"].T + (ws["p.down.b"] if bias else 0)
        x = rt.stream(torch.zeros(T, width, device=rt.device))
        part.forward(_t(f, rt.device, dtype), x, None)
        assert np.abs(x.data.cpu().numpy() - want).max() < _tol(dtype) * np.abs(want).max(), T


# ------------------------------------------------------------------------------------------ attention, this design's
def _mixer(m, rt, E, eps):
    import cuca_b200.models.model  # noqa: F401  (registers the parts)
    from cuca_b200.config.pafutar_config import KeyValueAttentionConfig
    from cuca_b200.models.pafutar import _mixer_spec
    from cuca_b200.parts.base import MIXERS
    spec = _mixer_spec(KeyValueAttentionConfig.from_json(m, "mixer"), E, eps, "l0.mix.")
    return MIXERS.get(spec.kind)(spec, rt)


def _weights_for(part, seed):
    rs = np.random.default_rng(seed)
    return {name: pu.bf16_round(np.asarray(pu.draw(name, need, rs), dtype=np.float32)) for name, need in part.tensors().items()}


def _load(part, ws, rt):
    needs = part.tensors()
    part.load(lambda n: _t(ws[n], rt.device, torch.float32 if needs[n].keep_fp32 else rt.dtype))


class _Cache:
    """Pages in a scrambled order; before they are written they hold NaN (32-bit) or a large number. Pages behind a
    request's window may be taken away as the engine does."""

    def __init__(self, part, rt, bs, lengths, slots, seed=0):
        kv = part.cache_needs().kv
        self.bs, self.kv = bs, kv
        per = [-(-n // bs) for n in lengths]
        order = np.random.default_rng(seed).permutation(sum(per) + 3).tolist()
        shape = (sum(per) + 3, kv.n_kv_heads, bs)
        fill = float("nan") if rt.dtype == torch.float32 else 0.0
        self.k = torch.full((*shape, kv.head_dim), fill, dtype=rt.dtype, device=rt.device)
        self.v = None if kv.v_head_dim == 0 else torch.full((*shape, kv.v_head_dim or kv.head_dim), fill, dtype=rt.dtype, device=rt.device)
        self.key_scale = torch.full(shape, float("nan"), device=rt.device) if kv.key_scale else None
        table = np.full((max(slots) + 2, max(per) + 2), -1)
        for n, s in zip(per, slots):
            table[s, :n] = [order.pop() for _ in range(n)]
        self.full = table
        self.tables = torch.tensor(table, dtype=torch.int32, device=rt.device)

    def give_back(self, slot, length):
        """What the pools do once `length` positions are cached."""
        if self.kv.window is None:
            return
        upto, kept = max(0, length - (self.kv.window - 1)) // self.bs, -(-self.kv.keep_first // self.bs)
        if upto > kept:
            self.tables[slot, kept:upto] = -1

    def view(self, step):
        from cuca_b200.cache.device import CacheView
        return CacheView(self.k, self.v, self.tables, self.bs, 0, None, step.slots, self.key_scale)


def _run_attention(part, rt, cache, xs, cuts, slots, E, dtype):
    def fwd(h, step):
        out = rt.stream(torch.zeros(h.shape[0], E, device=rt.device))
        part.forward(h.to(dtype), out, step, cache.view(step))
        data = out.data.clone()
        for s, a, n in zip(step.host["slots"], step.host["starts"], step.host["counts"]):
            cache.give_back(s, a + n)
        return data
    got = _run_cut(rt.device, fwd, xs, cuts, slots, E)
    assert int(rt.err.item()) == 0
    return got


ATTENTIONS = [pu.attn(), pu.attn(heads=3, kv_heads=3, dim=8, window=5, keep=1), pu.attn(heads=1, kv_heads=1, dim=20, window=1, keep=0),
              pu.attn(heads=5, kv_heads=1, dim=12, scale=None, window=None), pu.attn(heads=6, kv_heads=2, dim=64, window=24, keep=2),
              pu.attn(heads=2, kv_heads=1, dim=128, window=9, keep=70), pu.attn(heads=16, kv_heads=1, dim=16, window=40, keep=17),
              pu.attn(heads=4, kv_heads=4, dim=32, window=64, keep=0), pu.attn(heads=8, kv_heads=2, dim=48, window=30, keep=4),
              pu.attn(heads=3, kv_heads=1, dim=128, window=None), pu.attn(heads=4, kv_heads=2, dim=136, window=17, keep=3)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bs", [8, 16])
@pytest.mark.parametrize("m", ATTENTIONS)
def test_attention_alone_whole_and_cut(dtype, bs, m):
    rt, E, eps = _rt(dtype), 40, 1e-5
    part = _mixer(m, rt, E, eps)
    ws = _weights_for(part, 7)
    _load(part, ws, rt)
    rs = np.random.default_rng(8)
    xs = [pu.bf16_round(rs.normal(0, 1.5, (n, E))) for n in (151, 20, 83)]
    want = [pp.attention(x, ws, "l0.mix.", m, eps) for x in xs]
    for cuts in ([CUTS[0]] * 3, [CUTS[1], CUTS[2], CUTS[1]], [[2, 3, 60, 2, 63, 1000], CUTS[1], [80, 1, 1, 1]], [[1] * 151, [19, 1], [1] * 83]):
        cache = _Cache(part, rt, bs, [len(x) for x in xs], [2, 0, 3])
        got = _run_attention(part, rt, cache, xs, cuts, [2, 0, 3], E, dtype)
        for a, b in zip(got, want):
            assert np.abs(a - b).max() < _tol(dtype) * max(1.0, np.abs(b).max()), cuts


@pytest.mark.parametrize("eps", [1e-6, 0.3])
def test_unit_norm_and_page_write(eps):
    """The kernel between projection and attention: q normed and multiplied in place, k normed into its page, the raw k (or
    the row's own v) as value; the 16-bytes-a-lane form, the general one (unaligned rows, odd head sizes) and 32-bit."""
    from cuca_b200.kernels import ops
    for dtype in DTYPES:
        rt = _rt(dtype)
        dev = rt.device
        for nh, nkv, d, own_v, pad in ((6, 2, 64, False, 0), (3, 3, 40, False, 0), (4, 1, 256, True, 8), (5, 1, 20, False, 0), (2, 2, 64, True, 3), (1, 1, 8, False, 16)):
            rs = np.random.default_rng(d + nh)
            cols = (nh + nkv * (2 if own_v else 1)) * d + pad
            rows, bs = 21, 8
            src = pu.bf16_round(rs.normal(0, 1, (rows, cols)))
            src[4, :d] = 0.0  # a query of nothing stays nothing
            proj = _t(src, dev, dtype)
            mul = rs.uniform(-2, 2, nh)
            step = _step(dev, [(5, 13), (30, 1), (0, 7)], [1, 0, 2])
            tables = torch.full((3, 4), -1, dtype=torch.int32, device=dev)
            tables[1, :3], tables[0, 3], tables[2, 0] = torch.tensor([7, 2, 5], dtype=torch.int32), 0, 6
            k = torch.zeros(8, nkv, bs, d, dtype=dtype, device=dev)
            v = torch.zeros(8, nkv, bs, d, dtype=dtype, device=dev)
            v_col = (nh + nkv) * d if own_v else nh * d
            ops.norm_rope_store(proj, nh * d, v_col, step.positions, step.seq_of_row, tables, None, None, 0, False, None, None, False,
                                eps, k, v, bs, nh, nkv, d, d, rt.err, unit=True, q_mul=_t(mul, dev))
            # one row for both, and the norm's factor beside it
            again, k1, f1 = _t(src, dev, dtype), torch.zeros_like(k), torch.zeros(8, nkv, bs, device=dev)
            ops.norm_rope_store(again, nh * d, nh * d, step.positions, step.seq_of_row, tables, None, None, 0, False, None, None, False,
                                eps, k1, None, bs, nh, nkv, d, d, rt.err, unit=True, q_mul=_t(mul, dev), key_scale=f1)
            assert torch.equal(again, proj)
            tol = 1e-5 if dtype == torch.float32 else 1e-2
            q = src[:, :nh * d].reshape(rows, nh, d)
            want = pp.rms(q, eps) * mul[:, None]
            got = proj.float().cpu().numpy()
            assert np.abs(got[:, :nh * d].reshape(want.shape) - want).max() < tol * np.abs(want).max()
            assert np.array_equal(got[:, nh * d:], src[:, nh * d:].astype(np.float32))
            tb = tables.cpu().numpy()
            for r, (p, s) in enumerate(zip(step.positions.tolist(), step.seq_of_row.tolist())):
                kk, vv = src[r, nh * d:(nh + nkv) * d].reshape(nkv, d), src[r, v_col:v_col + nkv * d].reshape(nkv, d)
                at = (tb[s, p // bs], slice(None), p % bs)
                assert np.abs(k[at].float().cpu().numpy() - pp.rms(kk, eps)).max() < tol * 8
                assert np.array_equal(v[at].float().cpu().numpy(), vv.astype(np.float32))
                assert np.array_equal(k1[at].float().cpu().numpy(), kk.astype(np.float32))
                assert np.allclose(f1[at].cpu().numpy(), 1 / np.sqrt(np.mean(kk * kk, axis=1) + eps), rtol=1e-5)
            assert int(rt.err.item()) == 0 and int((f1 != 0).sum()) == 21 * nkv


def _planted(dtype, m, n, far, askers, E=40, eps=1e-6):
    """A part and an input with one key that stands out: the last dimension of every query head reads input column 0, of
    every key head input column 1; only position `far` has column 1 set, only the rows `askers` column 0, and the heads'
    factors make the planted score 24 above the distance bias at the asker, while no other key has that dimension."""
    rt = _rt(dtype)
    part = _mixer(m, rt, E, eps)
    ws = _weights_for(part, 3)
    H, G, d, p = m["heads"], m["kv_heads"], m["dim"], "l0.mix."
    slope = np.array(pp.slopes(H))
    for a in range(H):
        ws[p + "q"][a * d + d - 1] = 0.0
        ws[p + "q"][a * d + d - 1, 0] = 40.0
        ws[p + "q.b"][a * d + d - 1] = 0.0
    for g in range(G):
        ws[p + "k"][g * d + d - 1] = 0.0
        ws[p + "k"][g * d + d - 1, 1] = 40.0
        ws[p + "k.b"][g * d + d - 1] = 0.0
    ws[p + "q"][:, 1] = 0.0
    dist = max(i - far for i in askers)
    # (the plain scores are about N(0, 1) times factor times scale times sqrt(d): kept well below the planted one)
    ws[p + "temp"] = pu.bf16_round((24.0 + slope * dist) / (d * m["scale"]))
    _load(part, ws, rt)
    x = np.random.default_rng(4).normal(0, 0.5, (n, E))
    x[:, :2] = 0.0
    x[far, 1] = 1.0
    x[list(askers), 0] = 1.0
    return rt, part, ws, pu.bf16_round(x)


EDGES = [(d, w, keep, far, n) for d in (16, 24, 64, 128) for w, keep, far, n in (
    (7, 0, 3, 40), (16, 3, 20, 60), (33, 16, 16, 80), (33, 17, 16, 80), (64, 5, 40, 150), (65, 4, 4, 110), (130, 1, 0, 300), (130, 2, 70, 300),
    (100, 64, 63, 330), (100, 64, 64, 330), (40, 130, 129, 340), (40, 130, 130, 340), (300, 8, 7, 420), (2, 1, 0, 140))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d, window, keep, far, n", EDGES)
def test_a_planted_key_at_the_edges_of_the_window_and_of_the_kept_keys(dtype, d, window, keep, far, n):
    """The rows just inside and just outside the window of a key that takes nearly all weight where it is seen, whole,
    decoded and with a cut between; a kept key is seen from far away, the first one that is not kept only in its window."""
    m = pu.attn(heads=4, kv_heads=2, dim=d, scale=1.0, window=window, keep=keep)
    kept = far < keep
    askers = sorted({i for i in (far + window - 2, far + window - 1, far + window, far + window + 1, n - 1) if far < i < n})
    rt, part, ws, x = _planted(dtype, m, n, far, askers)
    want = pp.attention(x, ws, "l0.mix.", m, 1e-6)
    # the planted key decides: a window one longer, or one kept key fewer or more, is far off at these rows
    other = dict(m, mask={"size": window, "keep_first": far} if kept else {"size": window + 1, "keep_first": keep})
    moved = np.abs(pp.attention(x, ws, "l0.mix.", other, 1e-6) - want).max(axis=1)
    assert moved[far + window] > 0.2 * np.abs(want).max()
    edge = far + window
    for cuts in ([1000], [max(1, edge - 3)] + [1] * (n - max(1, edge - 3)), [edge - 1, 2, 2, 1000], [edge, 2, 1000]):
        for bs in (16, 8):
            cache = _Cache(part, rt, bs, [n], [1])
            got = _run_attention(part, rt, cache, [x], [cuts], [1], x.shape[1], dtype)[0]
            err = np.abs(got - want).max(axis=1)
            assert err[askers].max() < _tol(dtype) * np.abs(want).max(), cuts
            if dtype == torch.float32:  # (the factors make the other rows' softmax too sharp for 16-bit queries)
                assert err.max() < 3 * _tol(dtype) * np.abs(want).max(), cuts


# ------------------------------------------------------------------------------------------ attention, the kernels' options
def _plain_options(q, k, v, o):
    """Scores with cap, distance bias, window, kept keys, sink and gate in 64-bit, row by row; q: [T, H, d]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        js = pp.visible(t, {"size": o["window"], "keep_first": o["keep"]} if o["window"] else None)
        for a in range(H):
            s = (k[js, a // (H // G)] @ q[t, a]) * o["scale"]
            if o["cap"]:
                s = o["cap"] * np.tanh(s / o["cap"])
            if o["slopes"] is not None:
                s = s - o["slopes"][a] * (t - js)
            top = max(s.max(), o["sink"][a]) if o["sink"] is not None else s.max()
            e = np.exp(s - top)
            out[t, a] = (e / (e.sum() + (np.exp(o["sink"][a] - top) if o["sink"] is not None else 0.0))) @ v[js, a // (H // G)]
    if o["gate"] is not None:
        out = out * pp.sigmoid(o["gate"])
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [24, 32, 64, 128])
@pytest.mark.parametrize("one_row", [False, True])
@pytest.mark.parametrize("window, keep, cap, slopes, sink, gate", [
    (None, 0, 0.0, True, False, False), (50, 3, 3.0, True, True, True), (90, 0, 0.0, False, False, False), (130, 66, 0.0, False, True, False), (300, 20, 5.0, True, False, True),
    (None, 0, 2.0, True, True, True), (20, 200, 0.0, True, False, True)])
def test_attention_options_in_every_form(dtype, d, window, keep, cap, slopes, sink, gate, one_row):
    """Every option with every other, rows of keys and values apart or one row for both with a factor per key, through the plain kernel, the two prompt forms and the split-key decode form (one
    chunk, several merged as a cluster, several through memory); positions up to 600; pages the window has passed gone."""
    from cuca_b200.cache.device import CacheView
    from cuca_b200.kernels import ops
    rt = _rt(dtype)
    dev, H, G, T, bs = rt.device, 6, 2, 600, 16
    rs = np.random.default_rng(d)
    r = lambda *s: pu.bf16_round(rs.normal(0, 1, s))  # noqa: E731
    q, k, v = r(T, H, d), r(T, G, d), r(T, G, d)
    o = {"window": window, "keep": keep, "scale": 1.7 * d ** -0.5, "cap": cap, "slopes": rs.uniform(0.0, 0.1, H) if slopes else None,
         "sink": rs.normal(0, 2, H) if sink else None, "gate": r(T, H, d) if gate else None}
    factors = rs.uniform(0.2, 2.0, (T, G)).astype(np.float32)
    want = _plain_options(q, k * factors[:, :, None] if one_row else k, k if one_row else v, o)
    order = rs.permutation(T // bs + 2)[:-(-T // bs)]
    kp, vp = torch.zeros(T // bs + 2, G, bs, d, dtype=dtype, device=dev), torch.zeros(T // bs + 2, G, bs, d, dtype=dtype, device=dev)
    pos = np.arange(T)
    kp[order[pos // bs], :, pos % bs] = _t(k, dev, dtype)
    vp[order[pos // bs], :, pos % bs] = _t(v, dev, dtype)
    tables = torch.full((2, T // bs + 4), -1, dtype=torch.int32, device=dev)
    tables[1, :len(order)] = torch.tensor(order, dtype=torch.int32)
    opts = {"softcap": cap, "slopes": None if o["slopes"] is None else _t(o["slopes"], dev), "keep_first": keep, "sink": sink,
            "sink_values": None if o["sink"] is None else _t(o["sink"], dev)}
    if one_row:
        vp, opts["key_scale"] = kp, torch.full((T // bs + 2, G, bs), float("nan"), device=dev)
        opts["key_scale"][order[pos // bs], :, pos % bs] = _t(factors, dev)

    def run(rows, step, plan):
        qq = _t(q[rows].reshape(len(rows), -1), dev, dtype)
        out = torch.empty(len(rows), H * d, dtype=dtype, device=dev)
        gates = None if o["gate"] is None else _t(o["gate"][rows].reshape(len(rows), -1), dev, dtype)
        cache = CacheView(kp, vp, tables, bs, 0, None, step.slots)
        ops.attention(qq, out, cache, step, plan, H, G, d, o["scale"], window, rt.err, gate=gates, **opts)
        return out.float().cpu().numpy().reshape(len(rows), H, d)

    def check(got, rows):
        assert np.abs(got - want[rows]).max() < (2e-5 if dtype == torch.float32 else 2e-2) * np.abs(want).max()
    for a, n in ((0, T), (0, 130), (70, 2), (129, 300), (517, 83)):
        if window and a > window:  # behind the first row's window and the kept keys there are no pages
            lo, hi = -(-keep // bs), (a - (window - 1)) // bs
            saved = tables.clone()
            tables[1, lo:max(lo, hi)] = -1
        step, rows = _step(dev, [(a, n)], [1]), np.arange(a, a + n)
        check(run(rows, step, ops.attention_plan(step)), rows)
        if dtype == torch.bfloat16:
            ops.USE_TC_ATTENTION = False
            try:
                check(run(rows, step, ops.attention_plan(_step(dev, [(a, n)], [1]))), rows)
            finally:
                ops.USE_TC_ATTENTION = True
        if window and a > window:
            tables.copy_(saved)
    for p in (0, 1, 15, 63, 64, 65, 130, 319, 320, 599):
        step = _step(dev, [(p, 1)], [1])
        plan = ops.attention_plan(step)
        check(run(np.array([p]), step, plan), [p])
        if dtype == torch.bfloat16 and d != 24:
            for chunk, n_splits in ((0, 1), (0, 4), (0, 8), (0, 7), (64, 10), (128, 5)):
                plan.chunk = lambda *args, c=(chunk, n_splits): c  # noqa: B023
                check(run(np.array([p]), step, plan), [p])
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("H, G, d", [(6, 2, 64), (2, 1, 128), (16, 1, 16), (4, 4, 32), (8, 1, 128)])
@pytest.mark.parametrize("gate, own_v, mul", [(True, False, True), (False, False, False), (True, True, True)])
def test_decode_that_makes_its_own_queries_and_keys(H, G, d, gate, own_v, mul):
    """The one-launch decode step fed by a projection's K slices against the plain equations: norms, factors, page write,
    distance bias, window with kept keys, gate; one chunk and several, values that are the keys and values of their own."""
    from cuca_b200.cache.device import CacheView
    from cuca_b200.kernels import ops
    rt = _rt(torch.bfloat16)
    dev, eps, bs, T = rt.device, 1e-4, 16, 420
    rs = np.random.default_rng(H + d)
    n_v = G if own_v else 0
    cols = (H + G + n_v + (H if gate else 0)) * d
    v_col, g_col = (H + G if own_v else H) * d, (H + G + n_v) * d
    bias, factor = pu.bf16_round(rs.normal(0, 0.5, cols)), rs.uniform(-1.5, 1.5, H) if mul else None
    slopes = rs.uniform(0, 0.05, H)
    for window, keep in ((None, 0), (100, 5), (33, 70)):
        ks, vs = pu.bf16_round(rs.normal(0, 1, (2, T, G, d))), pu.bf16_round(rs.normal(0, 1, (2, T, G, d)))
        lengths, slots = [5, 200, T - 1, 0], [3, 0, 2, 1]
        pages = -(-T // bs)
        kp, vp = torch.zeros(4 * pages, G, bs, d, dtype=torch.bfloat16, device=dev), torch.zeros(4 * pages, G, bs, d, dtype=torch.bfloat16, device=dev)
        tables = torch.tensor(rs.permutation(4 * pages).reshape(4, pages), dtype=torch.int32, device=dev)
        tb = tables.cpu().numpy()
        fp = torch.full((4 * pages, G, bs), float("nan"), device=dev)
        raw = rs.normal(0, 1, (5, 4, cols))
        total = raw.sum(0) + bias
        want = np.zeros((4, H, d))
        for r, (n, s) in enumerate(zip(lengths, slots)):
            k, v, at = ks[r % 2, :n], vs[r % 2, :n], np.arange(n)
            if not own_v:  # the page holds the values, which are the keys before their factors
                f = rs.uniform(0.3, 2.0, (n, G)).astype(np.float32)
                k = v * f[:, :, None]
                fp[tb[s, at // bs], :, at % bs] = _t(f, dev)
            kp[tb[s, at // bs], :, at % bs] = _t(k if own_v else v, dev, torch.bfloat16)
            vp[tb[s, at // bs], :, at % bs] = _t(v, dev, torch.bfloat16)
            q = pp.rms(total[r, :H * d].reshape(H, d), eps) * (factor[:, None] if mul else 1.0)
            kn = total[r, H * d:(H + G) * d].reshape(1, G, d)
            vn = total[r, v_col:v_col + G * d].reshape(1, G, d)
            o = {"window": window, "keep": keep, "scale": 0.4, "cap": 0.0, "slopes": slopes, "sink": None, "gate": None}
            kk, vv = np.concatenate([k, pp.rms(kn, eps)]), pu.bf16_round(np.concatenate([v, vn]))
            qq = np.zeros((n + 1, H, d))
            qq[n] = pu.bf16_round(q)
            js = pp.visible(n, {"size": window, "keep_first": keep} if window else None)
            for a in range(H):
                sc = kk[js, a // (H // G)] @ qq[n, a] * 0.4 - slopes[a] * (n - js)
                e = np.exp(sc - sc.max())
                want[r, a] = (e / e.sum()) @ vv[js, a // (H // G)]
            if gate:
                want[r] *= pp.sigmoid(total[r, g_col:].reshape(H, d))
            assert o["window"] == window
        step = _step(dev, [(n, 1) for n in lengths], slots)
        for chunk, n_splits in ((0, 1), (0, 2), (0, 4), (0, 8), (0, 6), (64, 8)):
            cache = CacheView(kp.clone(), vp.clone() if own_v else None, tables, bs, 0, None, step.slots, None if own_v else fp.clone())
            out = torch.empty(4, H * d, dtype=torch.bfloat16, device=dev)
            parts = ops.PartialSums(_t(raw, dev), 5)
            ops.attention_decode_fused_unit(parts, _t(bias, dev, torch.bfloat16), v_col, g_col if gate else None, eps,
                                            _t(factor, dev) if mul else None, out, cache, step, 4, H, G, d, 0.4, window, chunk,
                                            n_splits, rt.err, slopes=_t(slopes, dev), keep_first=keep,
                                            key_scale=cache.key_scale)
            got = out.float().cpu().numpy().reshape(4, H, d)
            assert np.abs(got - want).max() < 2e-2 * np.abs(want).max(), (window, chunk, n_splits)
            for r, (n, s) in enumerate(zip(lengths, slots)):
                row, key = cache.k[tb[s, n // bs], :, n % bs].float().cpu().numpy(), total[r, H * d:(H + G) * d].reshape(G, d)
                if not own_v:
                    assert np.abs(row - key).max() < 1e-2 * np.abs(row).max()
                    assert np.allclose(cache.key_scale[tb[s, n // bs], :, n % bs].cpu().numpy(), 1 / np.sqrt(np.mean(key * key, axis=1) + eps), rtol=1e-4)
                    continue
                assert np.abs(row - pp.rms(key, eps)).max() < 2e-2 * np.abs(row).max()
                row = cache.v[tb[s, n // bs], :, n % bs].float().cpu().numpy()
                assert np.abs(row - total[r, v_col:v_col + G * d].reshape(G, d)).max() < 1e-2 * np.abs(row).max()
    assert int(rt.err.item()) == 0


# ------------------------------------------------------------------------------------------ whole models
LENGTHS = {"mix": [1, 2, 5, 16, 33, 64, 97, 130], "plain": [3, 17, 48, 100], "one": [1, 18, 35, 77, 120],
           "wide": [1, 15, 33, 38, 76, 140, 230], "two": [2, 40, 90]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(pu.CONFIGS.items()):
        weights = pu.make_weights(cfg, seed=20 + i)
        out[name] = (pu.write_model(tmp_path_factory.mktemp(f"pafutar_{name}"), cfg, weights), cfg, pu.Oracle(cfg, weights))
    return out


def _requests(name, cfg):
    return {f"r{n}": pu.random_tokens(n, cfg["vocab"], seed=300 + n) for n in LENGTHS[name]}


def test_the_stream_after_every_layer(models):
    from cuca_b200.engine.core import EngineCore
    from cuca_b200.engine.step import StepEntry
    for name in pu.CONFIGS:
        folder, cfg, oracle = models[name]
        for dtype in ("float32", "bfloat16"):
            core = EngineCore.from_folder(folder, dtype=dtype, kv_tokens=128, context_length=128, window_pools="full")
            seen = []
            core.model.layer_hook = lambda n, stream: seen.append(stream.data.cpu().numpy().copy())
            toks = pu.random_tokens(29, cfg["vocab"], 4)
            blocks, slot = core.pools.new_seq(), core.slots.alloc()
            core.cache.clear_slot(slot)
            core.pools.reserve(blocks, len(toks))
            core.stepper.step([StepEntry(blocks, slot, toks, [0])])
            want = []
            pp.forward(cfg, oracle.w, toks, want)
            assert len(seen) == len(want) == len(cfg["layers"])
            for a, b in zip(seen, want):
                assert np.abs(a - b).max() < (1e-4 if dtype == "float32" else 6e-2) * np.abs(b).max(), (name, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(pu.CONFIGS))
def test_whole_and_decoded_one_by_one(models, name, dtype):
    folder, cfg, oracle = models[name]
    reqs = _requests(name, cfg)
    for steps in (ru.trace_whole(reqs), ru.trace_tail_one_by_one(reqs, tail=48)):
        got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=8)
        pu.compare(steps, got, reqs, oracle, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(pu.CONFIGS))
def test_portions_down_to_two_tokens(models, name, dtype):
    folder, cfg, oracle = models[name]
    reqs = _requests(name, cfg)
    for sizes in ((5, 2, 17, 3, 2, 32, 7, 2, 64, 11), (2, 2, 3, 1, 1, 8, 9, 40)):
        steps = ru.trace_portions(reqs, sizes=sizes)
        got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=16)
        pu.compare(steps, got, reqs, oracle, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(pu.CONFIGS))
def test_mixed_batches_reuse_pages_and_slots(models, name, dtype):
    """Eight and more requests through four (and three) slots and a pool sized for the peak (and, for windows, for the
    window and the kept pages): every slot and most pages serve several requests, whose state must start from zero."""
    folder, cfg, oracle = models[name]
    reqs = _requests(name, cfg)
    reqs.update({f"s{n}": pu.random_tokens(n, cfg["vocab"], seed=900 + n) for n in (4, 9, 23, 31, 58)})
    for live, pools in ((4, "full"), (3, "sized")):
        steps = ru.trace_mixed(reqs, max_live=live, seed=7 + live)
        got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=8, window_pools=pools)
        pu.compare(steps, got, reqs, oracle, dtype)


def test_32_bit_hardly_depends_on_cuts_or_company(models):
    folder, cfg, _ = models["mix"]
    reqs = {"a": pu.random_tokens(70, cfg["vocab"], 1), "b": pu.random_tokens(33, cfg["vocab"], 2)}
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
    """Three hundred tokens decoded one by one: every window fills and slides over decoded tokens, pages behind it come back
    and are used again, the kept pages stay."""
    folder, cfg, oracle = models["wide"]
    reqs = {"long": pu.random_tokens(330, cfg["vocab"], 5)}
    steps = ru.trace_tail_one_by_one(reqs, tail=300)
    for dtype in ("float32", "bfloat16"):
        got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=8, window_pools="sized")
        pu.compare(steps, got, reqs, oracle, dtype)


def test_long_prompts(models):
    for name in ("mix", "wide"):
        folder, cfg, oracle = models[name]
        reqs = {"p": pu.random_tokens(610, cfg["vocab"], 8), "q": pu.random_tokens(300, cfg["vocab"], 9)}
        for steps in (ru.trace_whole(reqs), ru.trace_portions(reqs, sizes=(7, 300, 2, 280, 1, 64))):
            for dtype in ("bfloat16", "float32"):
                got = ru.run_in_process(folder, dtype, steps, ru.peak_tokens(steps), block_size=16)
                pu.compare(steps, got, reqs, oracle, dtype)


def test_a_request_ends_where_the_learned_positions_do(models):
    """`max_positions` tokens run; one more is refused before anything happens."""
    from cuca_b200.engine.core import EngineCore
    from cuca_b200.engine.step import StepEntry, StepError
    folder, cfg, oracle = models["one"]
    n = cfg["max_positions"]
    toks = pu.random_tokens(n + 1, cfg["vocab"], 2)
    core = EngineCore.from_folder(folder, dtype="float32", kv_tokens=n + 32)
    assert core.context_length == n
    blocks, slot = core.pools.new_seq(), core.slots.alloc()
    core.cache.clear_slot(slot)
    core.pools.reserve(blocks, n)
    logits = core.stepper.step([StepEntry(blocks, slot, toks[:n], [n - 1])])
    want = oracle.logits("full", toks[:n])[-1]
    assert np.abs(logits[0].cpu().numpy() - want).max() < 1e-4 * np.abs(want).max()
    core.pools.reserve(blocks, n + 1)
    with pytest.raises(StepError):
        core.stepper.step([StepEntry(blocks, slot, toks[n:], [0])])
    core.rt.check_device_errors()


def test_trace_run_as_a_program(models):
    folder, cfg, oracle = models["one"]
    reqs = _requests("one", cfg)
    steps = ru.trace_mixed(reqs, max_live=4, seed=1)
    got = ru.run_subprocess(folder, "float32", steps, ru.peak_tokens(steps))
    pu.compare(steps, got, reqs, oracle, "float32")


# ------------------------------------------------------------------------------------------ the entry point
def _plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(pp.forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]


@pytest.mark.parametrize("name", ["mix", "plain"])
def test_greedy_generation_through_the_entry_point(models, name):
    """`LocalModel.generate`: the scheduler admits, cuts prompts into portions, decodes through captured graphs and gives
    slots to later requests; the tokens are the plain implementation's greedy ones."""
    from cuca_b200 import BatchingConfig, LocalModel, LocalModelConfig
    folder, cfg, oracle = models[name]
    prompts = [pu.random_tokens(n, cfg["vocab"], seed=40 + n) for n in (3, 50, 21, 9, 70)]
    model = LocalModel.load(LocalModelConfig(source=str(folder), dtype="float32", context_length=256,
                                             batching=BatchingConfig(max_sequences=2, prefill_chunk=16)))
    outs = model.generate(prompts, max_tokens=12, temperature=0.0)
    for prompt, out in zip(prompts, outs):
        assert out.tokens == _plain_greedy(cfg, oracle.w, prompt, 12)


def test_a_prompt_longer_than_a_windows_pool_is_generated_from(models):
    """A prompt of many windows through pools that hold a window, the kept pages and one step's tokens."""
    from cuca_b200 import BatchingConfig, LocalModel, LocalModelConfig
    folder, cfg, oracle = models["two"]
    model = LocalModel.load(LocalModelConfig(source=str(folder), dtype="float32", context_length=256,
                                             batching=BatchingConfig(max_sequences=2, max_step_tokens=16, prefill_chunk=16)))
    assert all(g.n_blocks * model.core.block_size < 200 for g in model.core.groups)
    prompt = pu.random_tokens(230, cfg["vocab"], 3)
    assert model.generate(prompt, max_tokens=5, temperature=0.0).tokens == _plain_greedy(cfg, oracle.w, prompt, 5)


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
    prompt = pu.random_tokens(20, cfg["vocab"], 77)
    a = model.generate(prompt, max_tokens=16, temperature=1.0, top_k=20, seed=5).tokens
    b = model.generate(prompt, max_tokens=16, temperature=1.0, top_k=20, seed=5).tokens
    c = model.generate(prompt, max_tokens=16, temperature=1.0, top_k=20, seed=6).tokens
    assert a == b and a != c and all(0 <= t < cfg["vocab"] for t in a)
    with pytest.raises(StatefulCacheError):
        LocalModel.load(LocalModelConfig(source=str(folder), dtype="bfloat16", context_length=128,
                                         batching=BatchingConfig(prefix_cache=True)))


def test_bfloat16_generation_through_captured_graphs(models):
    """The serving precision end to end: prompts in portions, decode steps replayed as CUDA graphs (with padding rows: three
    requests in a bucket of four). Where two logits nearly tie bfloat16 may take the other branch, so every token it takes
    must be a near-maximum of the plain implementation's logits at its place."""
    from cuca_b200 import BatchingConfig, LocalModel, LocalModelConfig
    for name in ("two", "wide"):
        folder, cfg, oracle = models[name]
        prompts = [pu.random_tokens(n, cfg["vocab"], seed=60 + n) for n in (5, 70, 33)]
        model = LocalModel.load(LocalModelConfig(source=str(folder), dtype="bfloat16", context_length=256,
                                                 batching=BatchingConfig(max_sequences=4, prefill_chunk=32)))
        assert model.backend.use_graphs
        outs = model.generate(prompts, max_tokens=40, temperature=0.0)
        assert model.backend.graph_steps > 0
        for prompt, out in zip(prompts, outs):
            ref = pp.forward(cfg, oracle.w, prompt + out.tokens)
            for i, tok in enumerate(out.tokens):
                row = ref[len(prompt) - 1 + i]
                assert float(row.max() - row[tok]) < 0.06 * float(np.abs(row).max()), (name, i)
