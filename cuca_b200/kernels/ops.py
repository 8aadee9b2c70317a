"""Thin Python wrappers over the kernel library: tensors in, launches out.

Each function checks what the kernel cannot (device, dtype, contiguity) and
launches on torch's current stream. Nothing here computes on the host or falls
back to torch operators.
"""
from __future__ import annotations

import ctypes
import os

import torch

from . import library

F32, BF16 = 0, 1
EPI_STORE, EPI_RESIDUAL, EPI_SWIGLU = 0, 1, 2
_CODES = {torch.float32: F32, torch.bfloat16: BF16}


def dtype_code(dtype: torch.dtype) -> int:
    try:
        return _CODES[dtype]
    except KeyError:
        raise library.KernelError(f"kernels take float32 or bfloat16, not {dtype}") from None


_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)


def _stream() -> int:
    """The current stream's handle. Asked of torch's C entry where there is one: `torch.cuda.current_stream()` builds
    a Python object per call, 2.5 us of the 19 us of host time that a launch cost (a prompt step of a few tokens is
    230 launches whose kernels take 16 us each: the host set its pace)."""
    if _raw_stream is not None:
        return _raw_stream(torch.cuda.current_device())
    return torch.cuda.current_stream().cuda_stream


def _p(t):
    return None if t is None else t.data_ptr()


def _cuda(*tensors):
    for t in tensors:
        if t is not None and not t.is_cuda:
            raise library.KernelError("kernel arguments must live on the CUDA device (there is no CPU path)")


def embed(table: torch.Tensor, tokens: torch.Tensor, out: torch.Tensor, err: torch.Tensor, scale: float = 1.0) -> None:
    """out[r] = table[tokens[r]] * scale, into the 32-bit stream."""
    _cuda(table, tokens, out)
    lib = library.load()
    V, E = table.shape
    library.check(lib.cuca_embed_scaled(_p(table), dtype_code(table.dtype), _p(tokens), _p(out), tokens.shape[0], E, V,
                                        float(scale), _p(err), _stream()), "embed")


def embed_pos(table, pos_table, tokens, positions, out, err, scale: float = 1.0) -> None:
    """out[r] = table[tokens[r]] * scale + pos_table[positions[r]], into the 32-bit stream."""
    _cuda(table, pos_table, tokens, positions, out)
    V, E = table.shape
    library.check(library.load().cuca_embed_pos(_p(table), _p(pos_table), dtype_code(table.dtype), _p(tokens), _p(positions),
                                                _p(out), tokens.shape[0], E, V, pos_table.shape[0], float(scale), _p(err),
                                                _stream()), "embed_pos")


def embed_norm(table, tokens, out, weight, eps: float, err, scale: float = 1.0) -> None:
    """out[r] = e / sqrt(mean(e^2) + eps) * weight with e = table[tokens[r]] * scale, into the 32-bit stream."""
    _cuda(table, tokens, out, weight)
    V, E = table.shape
    library.check(library.load().cuca_embed_norm(_p(table), dtype_code(table.dtype), _p(tokens), _p(out), tokens.shape[0],
                                                 E, V, float(scale), _p(weight), float(eps), _p(err), _stream()),
                  "embed_norm")


def rmsnorm(x: torch.Tensor, weight: torch.Tensor, out: torch.Tensor, eps: float, rows=None, groups: int = 1) -> None:
    """out = x / sqrt(mean(x^2) + eps) * weight per row; `groups` > 1: every one of that many equal consecutive parts
    of a row is divided by its own root mean square."""
    _cuda(x, weight, out)
    lib = library.load()
    n = out.shape[0] if rows is None else rows.shape[0]
    library.check(lib.cuca_rmsnorm_groups(_p(x), _p(weight), dtype_code(weight.dtype), _p(out), dtype_code(out.dtype),
                                          _p(rows), n, x.shape[-1], float(eps), int(groups), _stream()), "rmsnorm")


def rope_store(qkv, positions, seq_of_row, tables, cos, sin, rotary_dim, kpool, vpool, block_size,
               n_heads, n_kv_heads, head_dim, err) -> None:
    """Rotate q (in place) and k, write k and v to their pages. `tables` is [S, width] int32;
    pools are [n_blocks, n_kv_heads, block_size, head_dim] (None with n_kv_heads == 0)."""
    _cuda(qkv, positions, seq_of_row)
    lib = library.load()
    n_blocks = kpool.shape[0] if kpool is not None else 0
    table_rows = cos.shape[0] if cos is not None else 0
    library.check(lib.cuca_rope_store(
        _p(qkv), dtype_code(qkv.dtype), _p(positions), _p(seq_of_row), _p(tables),
        tables.shape[1] if tables is not None else 0, _p(cos), _p(sin), table_rows, int(rotary_dim),
        _p(kpool), _p(vpool), n_blocks, int(block_size), qkv.shape[0], n_heads, n_kv_heads, head_dim,
        _p(err), _stream()), "rope_store")


def random_normal(out: torch.Tensor, key: int, first: int, mean: float, scale: float) -> None:
    """out.view(-1)[i] = mean + normal(key, first + i) * (2 * 65536 * scale): the counter-based generator of the
    random-weights mode (`weights/loader.py:host_normal` is its host form, bit for bit)."""
    _cuda(out)
    lib = library.load()
    library.check(lib.cuca_random_normal(_p(out), dtype_code(out.dtype), out.numel(), int(first), int(key),
                                         float(mean), float(scale), _stream()), "random_normal")


def swiglu(gate_up, out) -> None:
    _cuda(gate_up, out)
    lib = library.load()
    library.check(lib.cuca_swiglu(_p(gate_up), _p(out), dtype_code(out.dtype), out.shape[0], out.shape[1],
                                  _stream()), "swiglu")


def glu_capped(gate_up, out, limit: float, alpha: float) -> None:
    """out[r, j] = g sigmoid(alpha g) (u + 1), g = min(gate_up[r, j], limit), u = clamp(gate_up[r, ff + j], +-limit)."""
    _cuda(gate_up, out)
    library.check(library.load().cuca_glu_capped(_p(gate_up), _p(out), dtype_code(out.dtype), out.shape[0], out.shape[1],
                                                 float(limit), float(alpha), _stream()), "glu_capped")


GLU_SILU, GLU_GELU_TANH = 0, 1


def glu_act(gate_up, out, act: int) -> None:
    """out[r, j] = act(gate_up[r, j]) * gate_up[r, ff + j]; act: GLU_SILU or GLU_GELU_TANH."""
    _cuda(gate_up, out)
    library.check(library.load().cuca_glu_act(_p(gate_up), _p(out), dtype_code(out.dtype), out.shape[0], out.shape[1],
                                              int(act), _stream()), "glu_act")


def head_gate_(a, gate, n_heads: int, v_head_dim: int) -> None:
    """a[r, h * dv + j] *= sigmoid(gate[r, h]): one gate per head; both of one dtype, rows of any stride."""
    _cuda(a, gate)
    library.check(library.load().cuca_head_gate(_p(a), a.stride(0), _p(gate), gate.stride(0), dtype_code(a.dtype),
                                                a.shape[0], int(n_heads), int(v_head_dim), _stream()), "head_gate")


def softcap_(a, cap: float) -> None:
    """a <- cap tanh(a / cap) in place (32-bit)."""
    _cuda(a)
    if a.dtype != torch.float32 or not a.is_contiguous():
        raise library.KernelError("softcap_ takes a contiguous 32-bit tensor")
    library.check(library.load().cuca_softcap(_p(a), a.numel(), float(cap), _stream()), "softcap")


def add_to_stream(x, delta) -> None:
    _cuda(x, delta)
    lib = library.load()
    library.check(lib.cuca_add_to_stream(_p(x), _p(delta), dtype_code(delta.dtype), x.numel(), _stream()),
                  "add_to_stream")


def gemm_simt(a, w, out, epilogue=EPI_STORE, bias=None) -> None:
    """out = epilogue(a @ w.T) on CUDA cores; a: [M, K] (row stride >= K), w: [N or 2N, K]."""
    _cuda(a, w, out)
    lib = library.load()
    M, K = a.shape
    N = out.shape[1]
    library.check(lib.cuca_gemm_simt(_p(a), _p(w), _p(bias), _p(out), dtype_code(a.dtype), dtype_code(out.dtype),
                                     M, N, K, a.stride(0), out.stride(0), epilogue, _stream()), "gemm_simt")


class AttentionOptions(ctypes.Structure):
    """What the attention kernels take besides queries, pages and sizes (`csrc/attention_options.cuh`)."""

    _fields_ = [("scale", ctypes.c_float), ("window", ctypes.c_int), ("keep", ctypes.c_int), ("softcap", ctypes.c_float),
                ("sink", ctypes.c_int), ("gate_stride", ctypes.c_int), ("sink_val", ctypes.c_void_p),
                ("slopes", ctypes.c_void_p), ("gate", ctypes.c_void_p), ("key_scale", ctypes.c_void_p)]


def attention_options(n_heads, scale, window=None, softcap=0.0, sink=False, sink_values=None, keep_first=0, slopes=None,
                      gate=None, gate_width=None, key_scale=None) -> AttentionOptions:
    """`window` w: a query sees the last w keys, itself included, and with `keep_first` k the first k of its request as
    well (None: all keys). `softcap` c > 0: a scaled score s becomes c tanh(s / c). `slopes` (32-bit, one per query
    head): slope * distance is taken off a score. `sink`: every row's denominator holds one more exp(0) that has no
    value, or exp(sink_values[head]) (32-bit, one number per query head) when those are given. `gate` ([rows,
    gate_width], of the output's dtype): the result is multiplied by sigmoid(gate). `key_scale` ([pages, key heads, positions
    of a page], 32-bit): the values are the keys (the key pool is given as value pool too), and a score's q . k is
    multiplied by its key's number before anything else."""
    o = AttentionOptions()
    o.scale, o.window, o.softcap = float(scale), int(window or 0), float(softcap or 0.0)
    o.keep = int(keep_first or 0) if window else 0
    o.sink, o.sink_val = int(bool(sink)), _per_head(sink_values, n_heads, "a sink's scores")
    o.slopes = _per_head(slopes, n_heads, "distance slopes")
    if gate is not None:
        _cuda(gate)
        if gate.dim() != 2 or gate.stride(1) != 1 or (gate_width is not None and gate.shape[1] < gate_width):
            raise library.KernelError(f"an output gate is [rows, {gate_width}] with contiguous rows, not {tuple(gate.shape)}")
        o.gate, o.gate_stride = gate.data_ptr(), gate.stride(0)
    o.key_scale = _key_scale(key_scale)
    return o


def _key_scale(key_scale):
    if key_scale is None:
        return None
    if key_scale.dtype != torch.float32 or not key_scale.is_contiguous():
        raise library.KernelError("the factors of keys are contiguous 32-bit numbers")
    _cuda(key_scale)
    return key_scale.data_ptr()


def attention_generic(q, q_stride, out, kpool, vpool, positions, seq_of_row, tables, n_heads, n_kv_heads,
                      head_dim, scale, window, err) -> None:
    _cuda(q, out, kpool, vpool)
    lib = library.load()
    library.check(lib.cuca_attention_generic(
        _p(q), int(q_stride), _p(out), out.stride(0), dtype_code(out.dtype), _p(kpool), _p(vpool), kpool.shape[0],
        kpool.shape[2], _p(positions), _p(seq_of_row), _p(tables), tables.shape[1], out.shape[0], n_heads,
        n_kv_heads, head_dim, float(scale), int(window or 0), _p(err), _stream()), "attention_generic")


def argmax(logits, out) -> None:
    _cuda(logits, out)
    lib = library.load()
    library.check(lib.cuca_argmax(_p(logits), logits.stride(0), logits.shape[0], logits.shape[1], _p(out),
                                  _stream()), "argmax")


_scratch: dict = {}
WORKSPACE_BYTES = 48 << 20
N_COUNTERS = 1024


def gemm_scratch(device):
    """Split-K scratch of the tensor-core contraction: 32-bit partial tiles and per-tile arrival counters
    (zeroed once; the kernel leaves them zeroed)."""
    key = (device.type, device.index)
    if key not in _scratch:
        _scratch[key] = (torch.empty(WORKSPACE_BYTES // 4, dtype=torch.float32, device=device),
                         torch.zeros(N_COUNTERS, dtype=torch.int32, device=device))
    return _scratch[key]


_tc_supported: dict = {}


def gemm_tc_supported(a, w) -> bool:
    """Whether the tensor-core kernel takes this problem (the library's answer, remembered by what it depends on:
    K, the row stride, the operands' alignment and whether the problem is empty)."""
    pa, pw = a.data_ptr(), w.data_ptr()
    key = (a.shape[1], a.stride(0), pa & 15, pw & 15, a.shape[0] > 0, w.shape[0] > 0)
    ok = _tc_supported.get(key)
    if ok is None:
        lib = library.load()
        ok = _tc_supported[key] = bool(lib.cuca_gemm_tc_supported(pa, pw, a.shape[0], w.shape[0], a.shape[1], a.stride(0)))
    return ok


def gemm_tc(a, w, out, epilogue=EPI_STORE, bias=None, err=None, max_splits=16) -> None:
    """out = epilogue(a @ w.T) on the tcgen05 tensor cores; bf16 operands, K and the row stride multiples of 8."""
    _cuda(a, w, out)
    lib = library.load()
    M, K = a.shape
    N = out.shape[1]
    ws, counters = gemm_scratch(a.device)
    library.check(lib.cuca_gemm_tc(_p(a), _p(w), _p(bias), _p(out), dtype_code(out.dtype), M, N, K, a.stride(0),
                                   out.stride(0), epilogue, _p(ws), ws.numel() * 4, _p(counters), counters.numel(),
                                   int(max_splits), _p(err), _stream()), "gemm_tc")


ACT_RELU2 = 1  # `gemm_tc_act`


def gemm_tc_act(a, w, out, act: int, bias=None, err=None, max_splits=16) -> None:
    """out = act(a @ w.T + bias) as the contraction's epilogue, from the 32-bit sums; act: ACT_RELU2."""
    _cuda(a, w, out)
    M, K = a.shape
    ws, counters = gemm_scratch(a.device)
    library.check(library.load().cuca_gemm_tc_act(_p(a), _p(w), _p(bias), _p(out), dtype_code(out.dtype), M, out.shape[1], K,
                                                  a.stride(0), out.stride(0), int(act), _p(ws), ws.numel() * 4,
                                                  _p(counters), counters.numel(), int(max_splits), _p(err), _stream()),
                  "gemm_tc_act")


def gemm_tc_glu(a, w, out, limit: float, alpha: float, err=None, max_splits=16) -> None:
    """out = g' sigmoid(alpha g') (u' + 1) of [g | u] = a @ w.T (w: gate rows, then up rows), g' = min(g, limit),
    u' = clamp(u, -limit, limit): the capped gated unit as the contraction's epilogue, from the 32-bit sums."""
    _cuda(a, w, out)
    lib = library.load()
    M, K = a.shape
    ws, counters = gemm_scratch(a.device)
    library.check(lib.cuca_gemm_tc_glu(_p(a), _p(w), _p(out), M, out.shape[1], K, a.stride(0), out.stride(0),
                                       float(limit), float(alpha), _p(ws), ws.numel() * 4, _p(counters),
                                       counters.numel(), int(max_splits), _p(err), _stream()), "gemm_tc_glu")


def gemm_tc_glu_act(a, w, out, act: int, err=None, max_splits=16) -> None:
    """out = act(g) * u of [g | u] = a @ w.T (w: gate rows, then up rows) as the contraction's epilogue, from the
    32-bit sums; act: GLU_SILU or GLU_GELU_TANH."""
    _cuda(a, w, out)
    lib = library.load()
    M, K = a.shape
    ws, counters = gemm_scratch(a.device)
    library.check(lib.cuca_gemm_tc_glu_act(_p(a), _p(w), _p(out), M, out.shape[1], K, a.stride(0), out.stride(0),
                                           int(act), _p(ws), ws.numel() * 4, _p(counters), counters.numel(),
                                           int(max_splits), _p(err), _stream()), "gemm_tc_glu_act")


def gemm_tc_glu_experts(a, w, out, weights, run: int, cols: int, limit: float, limit_s: float, alpha: float, err=None,
                        max_splits=16) -> None:
    """`gemm_tc_glu` for routed experts of `run` output columns each (`cols` in all, `run` a multiple of 16) and a shared
    expert behind them: column n of row m times weights[m, n // run]; the shared one's times weights[m, cols // run], with
    cap `limit_s`."""
    _cuda(a, w, out, weights)
    M, K = a.shape
    ws, counters = gemm_scratch(a.device)
    library.check(library.load().cuca_gemm_tc_glu_experts(
        _p(a), _p(w), _p(out), M, out.shape[1], K, a.stride(0), out.stride(0), float(limit), float(limit_s), float(alpha),
        _p(weights), weights.stride(0), int(run), int(cols), _p(ws), ws.numel() * 4, _p(counters), counters.numel(),
        int(max_splits), _p(err), _stream()), "gemm_tc_glu_experts")


def gemm_pair_mode(mode: int) -> None:
    """When contractions over many tokens run as pairs of CTAs on one tile (`tcgen05.mma.cta_group::2`): 1 where
    the library's rule expects them to be faster, 0 never, 2 wherever they can (tests and measurements), -1 as the
    environment variable CUCA_GEMM_PAIR says."""
    library.load().cuca_gemm_pair_mode(int(mode))
    _partial_slices.clear()  # what was remembered of the library's choices depended on the mode
    _partial_max.clear()


def gemm(a, w, out, epilogue=EPI_STORE, bias=None, err=None) -> None:
    """out = epilogue(a @ w.T), on the kernel that fits dtype and shape: tensor cores for bfloat16
    (rows of 16-byte multiples), CUDA cores for the 32-bit path and for shapes the former refuses."""
    if a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and (bias is None or bias.dtype == torch.bfloat16) \
            and gemm_tc_supported(a, w):
        gemm_tc(a, w, out, epilogue, bias, err)
    else:
        gemm_simt(a, w, out, epilogue, bias)


class AttentionPlan:
    """How a step's rows are handed to the attention kernels, derived from the step's per-request description:
    requests that bring one token go to the split-key decode form (their row numbers; None when every row is
    one), longer portions in tiles of consecutive rows to a prefill form. The tile heights are the kernel
    library's; the lists are made on the device (`cuca_attention_plan`), the counts on the host from the same
    per-request counts. One plan serves every attention layer of a step; tiles of a height and the key chunking
    for a (key heads, head size) pair are made when first asked for."""

    def __init__(self, step):
        counts = step.host["counts"]
        self.step = step
        self.static = step.static_max_len is not None
        if self.static:
            self.n_decode, self.max_len = step.n_rows, step.static_max_len
            self.n_portions = 0
        else:
            starts = step.host["starts"]
            single = [s + 1 for c, s in zip(counts, starts) if c == 1]
            self.n_decode, self.max_len = len(single), max(single, default=1)
            self.n_portions = len(counts) - self.n_decode
        self.identity = self.n_portions == 0  # every row is a single token: decode rows are 0..rows-1
        self._counts = counts
        self._decode_rows = None
        self._tiles: dict = {}
        self._chunking: dict = {}

    @property
    def decode_rows(self):
        if self.identity or self.n_decode == 0:
            return None
        if self._decode_rows is None:
            self._make(tile_rows(0))  # the list of single rows comes with the first tiling asked for
        return self._decode_rows

    def tiles(self, rows_per_tile: int):
        """(first rows, row counts, number of tiles) of the portions cut into tiles of this height."""
        if rows_per_tile not in self._tiles:
            self._make(rows_per_tile)
        return self._tiles[rows_per_tile]

    def _make(self, rows_per_tile: int) -> None:
        step = self.step
        n_tiles = sum(-(-c // rows_per_tile) for c in self._counts if c > 1)
        want_rows = self._decode_rows is None and not self.identity and self.n_decode > 0
        buf = torch.empty(2 * n_tiles + (self.n_decode if want_rows else 0), dtype=torch.int32,
                          device=step.positions.device)
        row0, nrows, rows = buf[:n_tiles], buf[n_tiles:2 * n_tiles], buf[2 * n_tiles:]
        lib = library.load()
        library.check(lib.cuca_attention_plan(_p(step.req_row0), _p(step.req_count), _p(step.req_start), step.n_seqs,
                                              rows_per_tile, _p(rows) if want_rows else None,
                                              self.n_decode if want_rows else 0, _p(row0), _p(nrows), n_tiles,
                                              _stream()), "attention_plan")
        self._tiles[rows_per_tile] = (row0, nrows, n_tiles)
        if want_rows:
            self._decode_rows = rows

    def chunk(self, n_kv_heads: int, head_dim: int, window=None, keep_first: int = 0, one_row: bool = False):
        """(chunk, most chunks of a row) of the decode form; a window bounds the 64-key tiles that a row walks. `one_row`:
        a page row is key and value."""
        max_len = self.max_len
        if window:
            max_len = min(max_len, (-(-int(keep_first or 0) // 64) + -(-int(window) // 64) + 1) * 64)
        key = (n_kv_heads, head_dim, max_len, one_row)
        if key not in self._chunking:
            self._chunking[key] = decode_chunking(self.n_decode, n_kv_heads, max_len, head_dim, one_row=one_row)
        return self._chunking[key]


def attention_plan(step):
    """The step's plan for the attention kernels (made once per step), or None for a hand-made batch that carries
    no per-request description: such a batch runs through the plain kernel."""
    if getattr(step, "req_start", None) is None or "counts" not in step.host:
        return None
    plan = step.plans.get("paged_attention")
    if plan is None:
        plan = step.plans["paged_attention"] = AttentionPlan(step)
    return plan


_tile_rows: dict = {}


def tile_rows(which: int) -> int:
    """Rows per tile of a prefill form, asked of the kernel library: 0 the `mma.sync` form, 1 the tcgen05 form."""
    if which not in _tile_rows:
        _tile_rows[which] = int(library.load().cuca_attention_tile_rows(which))
    return _tile_rows[which]


_attn_scratch: dict = {}
_attn_scratch_retired: list = []  # superseded buffers: a captured graph may still hold their addresses
USE_TC_ATTENTION = True  # prompt portions through the tcgen05 attention where the shape allows


def attention_scratch(device, floats: int, counters: int):
    """Scratch of the split-key decode attention: partial (acc, max, sum) per chunk, arrival counters
    (zeroed once; the kernel leaves them zeroed). Grows (by doubling at least) when a step needs more. A captured
    graph keeps the addresses it was captured with, so a superseded buffer is never freed: replays of an older
    graph go on writing into memory that is still this module's, and its counters still start at zero."""
    key = (device.type, device.index)
    part, cnt = _attn_scratch.get(key, (None, None))
    if part is None or part.numel() < floats:
        if part is not None:
            _attn_scratch_retired.append(part)
        part = torch.empty(max(floats, 1 << 20, 2 * (part.numel() if part is not None else 0)), dtype=torch.float32,
                           device=device)
    if cnt is None or cnt.numel() < counters:
        if cnt is not None:
            _attn_scratch_retired.append(cnt)
        cnt = torch.zeros(max(counters, 4096, 2 * (cnt.numel() if cnt is not None else 0)), dtype=torch.int32,
                          device=device)
    _attn_scratch[key] = (part, cnt)
    return part, cnt


def attention_mma_supported(n_heads, n_kv_heads, head_dim, q_stride, out_stride) -> bool:
    lib = library.load()
    return bool(lib.cuca_attention_mma_supported(n_heads, n_kv_heads, head_dim, q_stride, out_stride))


_sms: dict = {}


def sm_count() -> int:
    """SMs of the current device, asked of the kernel library once per device."""
    dev = torch.cuda.current_device()
    if dev not in _sms:
        _sms[dev] = int(library.load().cuca_sm_count())
    return _sms[dev]


def decode_chunking(n_rows: int, n_kv_heads: int, max_len: int, head_dim: int = 128, sms: int | None = None,
                    one_row: bool = False):
    """(chunk, n_splits) of the decode attention. chunk 0: every row spreads its own keys evenly over the
    chunks it uses (the kernel repeats this choice per row from the row's own length, never above n_splits).
    n_splits minimises the time on the critical path in units of one 64-key tile: rounds of CTAs the GPU needs
    (a CTA holds three stages of a key and a value tile in shared memory) times (tiles per chunk + about three
    tiles' worth of fixed work per CTA); at most 32 and at most one chunk per tile of the longest row. A tile of rows that
    are key and value at once (`one_row`) takes half the time, so the fixed parts count double (8 rows of 1,055 keys, 4 key
    heads: 4 chunks as clusters 10.7 us, 9 through memory 11.8)."""
    if sms is None:
        sms = sm_count()
    tiles = max(1, -(-max_len // 64))
    forced = os.environ.get("CUCA_DECODE_SPLITS")  # a measuring aid: this many equal chunks for every row
    if forced:
        n = max(1, min(32, tiles, int(forced)))
        return -(-tiles // n) * 64, n
    slots = _decode_slots(head_dim, sms)
    pairs = max(1, n_rows * n_kv_heads)
    fixed, through_memory = (6, 26) if one_row else (3, 10)
    best, best_cost = 1, None
    for n in range(1, min(32, tiles) + 1):
        rounds = -(-pairs * n // slots)
        # the merge: none for one chunk, through distributed shared memory where a row's chunks run as a cluster,
        # through global memory and a last arriver else (measured: about a tile's time more, growing with the chunks)
        merge = 0 if n == 1 else 2 if _merge_as_cluster(pairs, n, slots) else through_memory + n // 2
        cost = rounds * (-(-tiles // n) + fixed) * 8 + merge
        if best_cost is None or cost < best_cost:
            best, best_cost = n, cost
    return 0, best


CLUSTER_MERGE = os.environ.get("CUCA_ATTN_CLUSTER", "1") != "0"
MAX_CLUSTER = 8  # the portable cluster size


def _decode_slots(head_dim: int, sms: int | None = None) -> int:
    """CTAs of the decode attention that are resident at once."""
    smem = 3 * 2 * 64 * (head_dim + 8) * 2 + 2048  # three stages of a key and a value tile
    return (sms or sm_count()) * max(1, min(8, (227 * 1024) // smem))


def _merge_as_cluster(pairs: int, n_splits: int, slots: int) -> bool:
    """Whether a row's chunk CTAs run as a thread-block cluster and merge through distributed shared memory. A
    cluster's CTAs keep their places until its slowest one has finished, a cluster lies within one GPC, and sizes
    that do not divide a GPC's places leave some empty: so only where every cluster is resident at once (clusters of
    two or four: the launch fits the GPU's places; of eight: half of them, since eight pack a GPC's places badly),
    and only for 2, 4 or 8 chunks. Measured: Llama-3.1-8B shape, batch 1, eight chunks: +1.3 % tokens/s as clusters;
    batch 8, 64 clusters of four (256 of 296 places): +0.5 %; batch 4, 32 clusters of eight (256 places): -9 %;
    Llama-2-13B shape, batch 8, 1,280 CTAs in five rounds: -11 %; batch 1, clusters of seven: -7 %."""
    return CLUSTER_MERGE and n_splits in (2, 4, 8) and pairs * n_splits * (2 if n_splits == 8 else 1) <= slots


def _decode_scratch(device, n_rows, n_heads, n_kv_heads, head_dim, n_splits):
    """Scratch of a split-key decode launch, or (None, None) when the row's chunk CTAs merge as a thread-block
    cluster through distributed shared memory: nothing then goes through global memory."""
    if n_splits == 1 or _merge_as_cluster(n_rows * n_kv_heads, n_splits, _decode_slots(head_dim)):
        return None, None
    return attention_scratch(device, n_rows * n_heads * n_splits * (head_dim + 2), n_rows * n_kv_heads)


def attention_decode(q, q_stride, out, kpool, vpool, positions, seq_of_row, tables, rows, n_rows, n_heads,
                     n_kv_heads, head_dim, scale, window, chunk, n_splits, err, **options) -> None:
    """The split-key decode form; `options`: see `attention_options`."""
    lib = library.load()
    part, cnt = _decode_scratch(out.device, n_rows, n_heads, n_kv_heads, head_dim, n_splits)
    opt = attention_options(n_heads, scale, window, gate_width=n_heads * head_dim, **options)
    library.check(lib.cuca_attention_decode_o(
        _p(q), int(q_stride), _p(out), out.stride(0), _p(kpool), _p(vpool), kpool.shape[0], kpool.shape[2],
        _p(positions), _p(seq_of_row), _p(tables), tables.shape[1], _p(rows), n_rows, n_heads, n_kv_heads, head_dim,
        ctypes.addressof(opt), chunk, n_splits, _p(part), _p(cnt), _p(err), _stream()), "attention_decode")


def _per_head(values, n_heads: int, what: str):
    """The pointer of one number per query head (None: null), checked for what the kernels assume."""
    if values is None:
        return None
    if values.dtype != torch.float32 or values.numel() != n_heads or not values.is_contiguous():
        raise library.KernelError(f"{what} are {n_heads} contiguous 32-bit numbers, one per query head")
    _cuda(values)
    return values.data_ptr()


def _sink_values(sink_values, n_heads: int):
    """The pointer of a sink's per-head scores (None: the sink's score is 0)."""
    return _per_head(sink_values, n_heads, "a sink's scores")


def attention_decode_fused(partial, bias, cos, sin, rotary_dim, has_kv, out, kpool, vpool, positions, seq_of_row, tables,
                           rows, n_rows, n_heads, n_kv_heads, head_dim, scale, window, chunk, n_splits, err) -> None:
    """The decode form fed by the stacked q/k/v projection's unadded K slices (`PartialSums`): adds them, rotates
    q and k, stores k and v in the pages and attends, in one launch. Every row of the step is a single token."""
    lib = library.load()
    part, cnt = _decode_scratch(out.device, n_rows, n_heads, n_kv_heads, head_dim, n_splits)
    library.check(lib.cuca_attention_decode_fused(
        _p(partial.data), partial.slices, partial.slice_stride, _p(bias), _p(cos), _p(sin),
        cos.shape[0] if cos is not None else 0, int(rotary_dim), int(bool(has_kv)), _p(out), out.stride(0), _p(kpool),
        _p(vpool), kpool.shape[0], kpool.shape[2], _p(positions), _p(seq_of_row), _p(tables), tables.shape[1], _p(rows),
        n_rows, n_heads, n_kv_heads, head_dim, float(scale), int(window or 0), chunk, n_splits, _p(part), _p(cnt),
        _p(err), _stream()), "attention_decode_fused")


def attention_decode_fused_unit(partial, bias, v_col, gate_col, eps, q_mul, out, cache, step, n_rows, n_heads, n_kv_heads,
                                head_dim, scale, window, chunk, n_splits, err, **options) -> None:
    """The decode form fed by a stacked projection's unadded K slices for layers without rotation whose queries and keys are
    divided by their root mean square per head: adds the slices, norms, multiplies the queries by `q_mul` (one factor per
    query head, or None), stores the page rows, attends and applies the output gate whose pre-activations stand at column
    `gate_col` (None: no gate), in one launch. Columns: q heads at 0, k heads behind them, v heads at `v_col` (with the option
    `key_scale` the k heads' column: the values are the keys as projected). Every row of the step is a single token."""
    part, cnt = _decode_scratch(out.device, n_rows, n_heads, n_kv_heads, head_dim, n_splits)
    opt = attention_options(n_heads, scale, window, **options)
    library.check(library.load().cuca_attention_decode_fused_unit(
        _p(partial.data), partial.slices, partial.slice_stride, _p(bias), partial.data.shape[2], int(v_col),
        -1 if gate_col is None else int(gate_col), float(eps), _per_head(q_mul, n_heads, "factors on the queries"), _p(out),
        out.stride(0), _p(cache.k), _p(cache.k if cache.v is None else cache.v), cache.k.shape[0], cache.k.shape[2], _p(step.positions),
        _p(step.seq_of_row), _p(cache.tables), cache.tables.shape[1], None, n_rows, n_heads, n_kv_heads, head_dim,
        ctypes.addressof(opt), chunk, n_splits, _p(part), _p(cnt), _p(err), _stream()), "attention_decode_fused_unit")


def attention_decode_fused_supported(plan, cache, out_dtype, n_rows, n_heads, n_kv_heads, head_dim) -> bool:
    """True when every row of the step is a single token of its request and the tensor-core decode form takes
    the shape: then rotate-and-store and attention are one launch."""
    bs = cache.block_size
    return (out_dtype == torch.bfloat16 and plan is not None and plan.identity and plan.n_decode == n_rows
            and n_rows > 0 and bs & (bs - 1) == 0 and head_dim % 16 == 0
            and attention_mma_supported(n_heads, n_kv_heads, head_dim, 2, n_heads * head_dim))


def attention_prefill(q, q_stride, out, kpool, vpool, positions, seq_of_row, tables, tile_row0, tile_nrows, n_tiles,
                      n_heads, n_kv_heads, head_dim, scale, window, err, **options) -> None:
    lib = library.load()
    opt = attention_options(n_heads, scale, window, gate_width=n_heads * head_dim, **options)
    library.check(lib.cuca_attention_prefill_o(
        _p(q), int(q_stride), _p(out), out.stride(0), _p(kpool), _p(vpool), kpool.shape[0], kpool.shape[2],
        _p(positions), _p(seq_of_row), _p(tables), tables.shape[1], _p(tile_row0), _p(tile_nrows), n_tiles, n_heads,
        n_kv_heads, head_dim, ctypes.addressof(opt), _p(err), _stream()), "attention_prefill")


def attention_tc_supported(q, out, kpool, vpool, n_heads, n_kv_heads, head_dim) -> bool:
    lib = library.load()
    return bool(lib.cuca_attention_tc_supported(n_heads, n_kv_heads, head_dim, kpool.shape[2], q.stride(0),
                                                out.stride(0), _p(q), _p(kpool), _p(vpool)))


# The largest head size the attention kernels take (`cuca_attention_max_head_dim` says the same; a constant here so
# that describing a model, as for writing a folder of random weights, does not need the kernel library).
ATTENTION_MAX_HEAD_DIM = 256


def attention_pair_tiles_mode(mode: int) -> None:
    """When a CTA of the tcgen05 prefill attention takes two tiles in turn (a heavy and a light one): 1 where that
    makes one round of CTAs out of more, 0 never, 2 whenever a launch has two tiles (tests), -1 as the environment
    variable CUCA_ATTN_PAIR_TILES says."""
    library.load().cuca_attention_pair_tiles_mode(int(mode))


def attention_prefill_tc(q, out, kpool, vpool, positions, seq_of_row, tables, tile_row0, tile_nrows, n_tiles,
                         n_heads, n_kv_heads, head_dim, scale, window, err, **options) -> None:
    """Prefill attention on tcgen05; tiles of up to 128 consecutive rows of one request."""
    lib = library.load()
    opt = attention_options(n_heads, scale, window, gate_width=n_heads * head_dim, **options)
    library.check(lib.cuca_attention_prefill_tc_o(
        _p(q), q.stride(0), q.shape[0], _p(out), out.stride(0), _p(kpool), _p(vpool), kpool.shape[0], kpool.shape[2],
        _p(positions), _p(seq_of_row), _p(tables), tables.shape[1], _p(tile_row0), _p(tile_nrows), n_tiles, n_heads,
        n_kv_heads, head_dim, ctypes.addressof(opt), _p(err), _stream()), "attention_prefill_tc")


def _gate_aligned(gate) -> bool:
    """Whether the tcgen05 attention takes this output gate (16 bytes a load)."""
    return gate is None or (gate.data_ptr() % 16 == 0 and gate.stride(0) % 8 == 0)


def attention(qkv, out, cache, step, plan, n_heads, n_kv_heads, head_dim, scale, window, err, **options) -> None:
    """Paged causal attention of every row of the step; q is the head of each `qkv` row. bfloat16 with head
    sizes 16..128 in steps of 16 runs on tensor cores: single-token requests through the split-key decode form,
    portions of prompts through the prefill form; everything else (the 32-bit path, other head sizes) through
    the plain kernel. `options` (cap, sink, kept first keys, distance bias, output gate): see `attention_options`."""
    bs = cache.block_size
    if (out.dtype == torch.bfloat16 and plan is not None and bs & (bs - 1) == 0
            and attention_mma_supported(n_heads, n_kv_heads, head_dim, qkv.stride(0), out.stride(0))):
        if plan.n_portions:
            if (USE_TC_ATTENTION and attention_tc_supported(qkv, out, cache.k, cache.v, n_heads, n_kv_heads, head_dim)
                    and _gate_aligned(options.get("gate"))):
                row0, nrows, n = plan.tiles(tile_rows(1))
                attention_prefill_tc(qkv, out, cache.k, cache.v, step.positions, step.seq_of_row, cache.tables,
                                     row0, nrows, n, n_heads, n_kv_heads, head_dim, scale, window, err, **options)
            else:
                row0, nrows, n = plan.tiles(tile_rows(0))
                attention_prefill(qkv, qkv.stride(0), out, cache.k, cache.v, step.positions, step.seq_of_row,
                                  cache.tables, row0, nrows, n, n_heads, n_kv_heads, head_dim, scale, window, err,
                                  **options)
        if plan.n_decode:
            chunk, n_splits = plan.chunk(n_kv_heads, head_dim, window, options.get("keep_first", 0),
                                         options.get("key_scale") is not None)
            attention_decode(qkv, qkv.stride(0), out, cache.k, cache.v, step.positions, step.seq_of_row,
                             cache.tables, plan.decode_rows, plan.n_decode, n_heads, n_kv_heads, head_dim, scale,
                             window, chunk, n_splits, err, **options)
        return
    attention_generic_v(qkv, qkv.stride(0), out, cache.k, cache.v, step.positions, step.seq_of_row, cache.tables,
                        n_heads, n_kv_heads, head_dim, head_dim, scale, window, err, **options)


def scatter_int(dst, idx, val) -> None:
    """dst.view(-1)[idx[i]] = val[i] on the device (page-table updates)."""
    _cuda(dst, idx, val)
    lib = library.load()
    library.check(lib.cuca_scatter_int(_p(dst), _p(idx), _p(val), idx.shape[0], dst.numel(), _stream()), "scatter_int")


def suppress_tokens(logits, ids) -> None:
    """logits[:, ids] = -inf on the device (`ids`: int32 tensor): tokens that must never be sampled."""
    _cuda(logits, ids)
    lib = library.load()
    library.check(lib.cuca_suppress_tokens(_p(logits), logits.stride(0), logits.shape[0], logits.shape[1], _p(ids),
                                           ids.shape[0], _stream()), "suppress_tokens")


def sample_scratch_words(vocab: int) -> int:
    n = 1
    while n < vocab:
        n <<= 1
    return n


class SampleSplit:
    """Scratch with which the greedy rows of a large vocabulary are cut over several CTAs each: per row the best of
    every part and a counter of the parts that have arrived (left zeroed by every launch). One per engine; a
    launch with more rows than it holds runs one CTA per row."""

    def __init__(self, rows: int, device):
        self.rows = int(rows)
        self.best = torch.zeros(self.rows * int(library.load().cuca_sample_max_split()), dtype=torch.int64, device=device)
        self.count = torch.zeros(self.rows, dtype=torch.int32, device=device)


def sample(logits, temperature, top_k, top_p, rng_state, slot_of_row, out, scratch=None, split: SampleSplit | None = None) -> None:
    """One token per row of `logits` [R, V] (32-bit). temperature/top_p: float32 [slots]; top_k: int32 [slots];
    rng_state: int64 [slots] SplitMix64 states, advanced for rows that draw; slot_of_row: int32 [R];
    scratch: int64 [R, words] for rows whose cut is wider than 1024 candidates (see `sample_scratch_words`)."""
    _cuda(logits, temperature, top_k, top_p, rng_state, slot_of_row, out)
    lib = library.load()
    library.check(lib.cuca_sample(_p(logits), logits.stride(0), logits.shape[0], logits.shape[1], _p(temperature),
                                  _p(top_k), _p(top_p), _p(rng_state), _p(slot_of_row), _p(out), _p(scratch),
                                  0 if scratch is None else scratch.shape[1],
                                  None if split is None else _p(split.best), None if split is None else _p(split.count),
                                  0 if split is None else split.rows, _stream()), "sample")


def decode_advance(tokens, positions, slot_of_row, sampled, history, counter, max_steps, err=None,
                   err_out=None) -> None:
    """tokens <- sampled, positions += 1 for live rows; history[counter] <- sampled; counter += 1;
    err_out[0] <- err[0] (the device error word rides along with the sampled tokens)."""
    lib = library.load()
    library.check(lib.cuca_decode_advance(_p(tokens), _p(positions), _p(slot_of_row), _p(sampled), _p(history),
                                          _p(counter), tokens.shape[0], int(max_steps), _p(err), _p(err_out),
                                          _stream()), "decode_advance")


# ------------------------------------------------------------------ partial sums (decode)
class PartialSums:
    """The result of a contraction over few tokens, left as K slices: `data` is [slices, rows, features] in
    32-bit; the kernel that reads it adds the slices in order (`add_partials_rmsnorm`, `rope_store_partial`)."""

    __slots__ = ("data", "slices")

    def __init__(self, data, slices):
        self.data, self.slices = data, slices

    @property
    def slice_stride(self) -> int:
        return self.data.stride(0)


_partial_max: list = []


def partial_max_tokens() -> int:
    """Most tokens for which a contraction may leave its K slices unadded (asked of the kernel library)."""
    if not _partial_max:
        _partial_max.append(int(library.load().cuca_gemm_tc_partial_max_tokens()))
    return _partial_max[0]


def _partial_plan(M: int, N: int, K: int, max_slices: int):
    """(slices, rows of a slice's slab) the library will use for this shape; slices 0: it does not take it."""
    key = (M, N, K, max_slices)
    plan = _partial_slices.get(key)
    if plan is None:
        lib = library.load()
        plan = _partial_slices[key] = (int(lib.cuca_gemm_tc_partial_slices(M, N, K, max_slices)),
                                       int(lib.cuca_gemm_tc_partial_rows(M, N)))
    return plan


def gemm_partial_supported(a, w) -> bool:
    return (a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and a.shape[0] <= partial_max_tokens()
            and gemm_tc_supported(a, w) and _partial_plan(a.shape[0], w.shape[0], a.shape[1], 16)[0] > 0)


_partial_slices: dict = {}  # (rows, features, K, most slices) -> (slices the kernel writes, rows of a slice's slab)
_slices_written = ctypes.c_int(0)  # where a launch reports how many it wrote
_SLICES_WRITTEN_AT = ctypes.addressof(_slices_written)


def gemm_partial(a, w, err=None, max_slices=16) -> PartialSums:
    """a @ w.T for few rows (`partial_max_tokens`), as partial sums over K slices (see `PartialSums`)."""
    _cuda(a, w)
    lib = library.load()
    M, K = a.shape
    N = w.shape[0]
    plan = _partial_plan(M, N, K, max_slices)
    slices, slab_rows = plan
    if slices <= 0:
        raise library.KernelError("gemm_partial: unsupported shape")
    # a slice's slab may be padded to the rows its kernel stores at once; the readers see [slices, M, N] of it
    data = torch.empty(slices, slab_rows, N, dtype=torch.float32, device=a.device)
    if slab_rows != M:
        data = data[:, :M]
    library.check(lib.cuca_gemm_tc_partial(_p(a), _p(w), _p(data), M, N, K, a.stride(0), max_slices,
                                           _SLICES_WRITTEN_AT, _p(err), _stream()), "gemm_partial")
    if _slices_written.value != slices:
        raise library.KernelError(f"gemm_partial: {_slices_written.value} slices written, {slices} expected")
    return PartialSums(data, slices)


def add_partials_rmsnorm(x, partial: PartialSums, weight, out, eps, rows=None, groups: int = 1) -> None:
    """x += sum of the slices (rows named by `rows`, else all); out = RMSNorm(x) * weight."""
    lib = library.load()
    n = out.shape[0]
    library.check(lib.cuca_add_partials_rmsnorm_groups(_p(x), _p(partial.data), partial.slices, partial.slice_stride,
                                                       _p(weight), _p(out), dtype_code(out.dtype), _p(rows), n,
                                                       x.shape[-1], float(eps), int(groups), _stream()),
                  "add_partials_rmsnorm")


def add_partials(x, partial: PartialSums) -> None:
    lib = library.load()
    library.check(lib.cuca_add_partials(_p(x), _p(partial.data), partial.slices, partial.slice_stride, x.numel(),
                                        _stream()), "add_partials")


# Most rows for which q/k/v are made from unadded slices: beyond, the rotate-and-store kernel that adds them (one
# block per row, every slice read again) costs more than the slices save (first token of a 300-token prompt on the
# Llama-3.1-8B shape: 7.9 ms that way, 7.4 ms with the projection written out and rotated in place).
ROPE_PARTIAL_MAX_ROWS = 256


def rope_store_partial(partial: PartialSums, bias, q_out, positions, seq_of_row, tables, cos, sin, rotary_dim, kpool,
                       vpool, block_size, n_heads, n_kv_heads, head_dim, err) -> None:
    lib = library.load()
    n_blocks = kpool.shape[0] if kpool is not None else 0
    table_rows = cos.shape[0] if cos is not None else 0
    library.check(lib.cuca_rope_store_partial(
        _p(partial.data), partial.slices, partial.slice_stride, _p(bias), _p(q_out), _p(positions), _p(seq_of_row),
        _p(tables), tables.shape[1] if tables is not None else 0, _p(cos), _p(sin), table_rows, int(rotary_dim),
        _p(kpool), _p(vpool), n_blocks, int(block_size), q_out.shape[0], n_heads, n_kv_heads, head_dim, _p(err),
        _stream()), "rope_store_partial")


# ------------------------------------------------------------------ blocks that norm a sublayer's input and output
def _gain(g):
    """(pointer, stride) of a norm's gain: a vector, or a single number for every coordinate."""
    return _p(g), (0 if g.numel() == 1 else 1)


def norm_shift(x, gain, eps, mix, kept, out, step) -> None:
    """out[r] = h[r] + (h[r-1] - h[r]) * mix, h = RMSNorm(x) * gain; the row before a request's first row of the step
    is `kept[slot]`, which then becomes the request's last h."""
    _cuda(x, gain, mix, kept, out)
    lib = library.load()
    gp, gs = _gain(gain)
    library.check(lib.cuca_norm_shift(_p(x), gp, gs, float(eps), _p(mix), _p(kept), _p(out), dtype_code(out.dtype),
                                      _p(step.seq_of_row), _p(step.req_row0), _p(step.req_count), _p(step.slots),
                                      x.shape[0], step.n_seqs, x.shape[1], _stream()), "norm_shift")


def post_norm_add(x, y, gain, eps, gain2=None, out=None) -> None:
    """x += RMSNorm(y) * gain; with `out`: out = RMSNorm(new x) * gain2 in the same pass."""
    _cuda(x, y, gain, out)
    lib = library.load()
    gp, gs = _gain(gain)
    g2p, g2s = _gain(gain2) if out is not None else (None, 0)
    library.check(lib.cuca_post_norm_add(_p(x), _p(y), gp, gs, g2p, g2s, _p(out),
                                         dtype_code(out.dtype) if out is not None else 0, x.shape[0], x.shape[1],
                                         float(eps), _stream()), "post_norm_add")


def gelu_(a, tanh_form: bool = False) -> None:
    """a = gelu(a) in place: the exact form (erf), or its tanh form."""
    _activation(a, 1 if tanh_form else 0)


def relu2_(a) -> None:
    """a = relu(a)^2 in place."""
    _activation(a, 2)


def _activation(a, form: int) -> None:
    _cuda(a)
    library.check(library.load().cuca_activation(_p(a), dtype_code(a.dtype), a.numel(), form, _stream()), "activation")


def scale_(a, s: float) -> None:
    _cuda(a)
    if a.dtype != torch.float32:
        raise library.KernelError("scale_ takes a 32-bit tensor")
    library.check(library.load().cuca_scale(_p(a), a.numel(), float(s), _stream()), "scale")


def concat2(a, b, out) -> None:
    """out[r] = [a[r] | b[r]] in out's dtype; a, b are 32-bit [rows, E]."""
    _cuda(a, b, out)
    library.check(library.load().cuca_concat2(_p(a), _p(b), _p(out), dtype_code(out.dtype), a.shape[0], a.shape[1],
                                              _stream()), "concat2")


# ------------------------------------------------------------------ recurrent mixers
MINGRU_CHUNK = 32  # tokens of a chunk where long portions run as chunks side by side
MINGRU_CHUNKED_FROM = 256  # portions at least this long, in the serving precision only


def mingru_scan(zxg, state, out, step) -> None:
    """The gated recurrence along every request's rows. Token by token in order (the 32-bit path always: its bits do
    not depend on how a prompt was cut); in bfloat16 a step with a long portion runs chunks of the portions side by
    side and carries the state across them in a short pass."""
    _cuda(zxg, state, out)
    counts = step.host.get("counts") if step.static_max_len is None else None
    if out.dtype == torch.bfloat16 and counts and max(counts) >= MINGRU_CHUNKED_FROM:
        max_chunks = -(-max(counts) // MINGRU_CHUNK)
        carry = torch.empty(step.n_seqs, max_chunks, 2, out.shape[1], dtype=torch.float32, device=out.device)
        library.check(library.load().cuca_mingru_scan_chunked(
            _p(zxg), _p(state), _p(carry), _p(out), dtype_code(out.dtype), _p(step.req_row0), _p(step.req_count),
            _p(step.slots), step.n_seqs, out.shape[1], MINGRU_CHUNK, max_chunks, _stream()), "mingru_scan_chunked")
        return
    library.check(library.load().cuca_mingru_scan(_p(zxg), _p(state), _p(out), dtype_code(out.dtype),
                                                  _p(step.req_row0), _p(step.req_count), _p(step.slots), step.n_seqs,
                                                  out.shape[1], _stream()), "mingru_scan")


def causal_conv(src, col0, weight, bias, kept, out, step) -> None:
    """out[r, c] = silu(bias[c] + sum_k weight[c, k] * src[r - (taps-1) + k, col0 + c]) along each request; inputs
    before a request's first row of the step come from `kept[slot]` ([taps - 1, C]), which is brought up to date."""
    _cuda(src, weight, kept, out)
    C, taps = weight.shape
    library.check(library.load().cuca_causal_conv(
        _p(src), src.stride(0), int(col0), _p(weight), _p(bias), dtype_code(weight.dtype), _p(kept), _p(out),
        _p(step.seq_of_row), _p(step.req_row0), _p(step.req_count), _p(step.slots), src.shape[0], step.n_seqs, C, taps,
        _stream()), "causal_conv")


def ssm_scan(xbc, proj, dt_col, dt_bias, a_log, d_skip, state, y, step, H, P, N, G) -> None:
    _cuda(xbc, proj, state, y)
    library.check(library.load().cuca_ssm_scan(
        _p(xbc), _p(proj), proj.stride(0), int(dt_col), _p(dt_bias), _p(a_log), _p(d_skip), _p(state), _p(y),
        _p(step.req_row0), _p(step.req_count), _p(step.slots), step.n_seqs, H, P, N, G, _stream()), "ssm_scan")


def gated_group_norm(y, z, weight, out, parts, eps) -> None:
    """out = RMSNorm over `parts` equal parts of (y * silu(z)) times weight; z: 32-bit rows of stride z.stride(0)."""
    _cuda(y, z, weight, out)
    library.check(library.load().cuca_gated_group_norm(
        _p(y), _p(z), z.stride(0), _p(weight), dtype_code(weight.dtype), _p(out), dtype_code(out.dtype), y.shape[0],
        y.shape[1], int(parts), float(eps), _stream()), "gated_group_norm")


# ------------------------------------------------------------------ attention over a cached latent
LATENT_MAX_RANK = 1024  # `cuca_latent_max_rank` says the same


def latent_prepare(qkg, H, dn, dr, rank, c_gain, eps, cos, sin, rot_dims, qk, cache, step, err,
                   half_pairs: bool = False) -> None:
    """Norms the latent, turns the shared key part and the heads' turned query parts by the row's position (pairs
    (2i, 2i + 1), or (i, i + rot_dims / 2) with `half_pairs`) and writes the cache row."""
    lib = library.load()
    pool = cache.k
    library.check(lib.cuca_latent_prepare_p(
        _p(qkg), qkg.stride(0), H, dn, dr, rank, _p(c_gain), float(eps), _p(cos), _p(sin), cos.shape[0], int(rot_dims),
        int(bool(half_pairs)), _p(qk), _p(pool), dtype_code(pool.dtype), pool.shape[0], pool.shape[2], _p(step.positions), _p(step.seq_of_row),
        _p(cache.tables), cache.tables.shape[1], qkg.shape[0], _p(err), _stream()), "latent_prepare")


def head_linear(a, lda, a_head, w, out, ldo, o_head, T, gate=None, ldg=0) -> None:
    """out[t, h, :] = w[h] @ a[t, h, :] for every head (w: [H, N, K]; a 32-bit), optionally times sigmoid(gate)."""
    H, N, K = w.shape
    library.check(library.load().cuca_head_linear(
        _p(a), int(lda), int(a_head), _p(w), dtype_code(w.dtype), _p(out), dtype_code(out.dtype), int(ldo), int(o_head),
        _p(gate), int(ldg), int(T), H, N, K, _stream()), "head_linear")


USE_MMA_LATENT = True  # bfloat16 caches through the tensor-core form where the sizes allow
LATENT_TILE_ROWS = 16  # tokens of a portion that one CTA of the tensor-core form takes
_latent_mma_ok: dict = {}


def latent_attention_mma_supported(rank: int, Dk: int) -> bool:
    key = (rank, Dk)
    if key not in _latent_mma_ok:
        _latent_mma_ok[key] = bool(library.load().cuca_latent_attention_mma_supported(rank, Dk))
    return _latent_mma_ok[key]


def latent_attention(qk, out, cache, step, H, rank, Dk, scale, window, err, sink_values=None) -> None:
    """Every row's heads attend over the cached rows of the row's request. A bfloat16 cache goes through the
    tensor-core form, portions of prompts in groups of 16 tokens per head and single tokens with their heads as the
    group (the step's attention plan names both); the 32-bit path and other sizes go through the plain kernel.
    `sink_values` (32-bit, one number per head): every denominator holds one more term exp(sink_values[head])."""
    pool = cache.k
    sink = _sink_values(sink_values, H)
    plan = attention_plan(step) if USE_MMA_LATENT and pool.dtype == torch.bfloat16 else None
    if plan is not None and latent_attention_mma_supported(rank, Dk):
        lib = library.load()

        def launch(row0, nrows, rows, n, splits=1, acc=None, ml=None):
            library.check(lib.cuca_latent_attention_mma_s(
                _p(qk), _p(out), _p(pool), pool.shape[0], pool.shape[2], _p(step.positions), _p(step.seq_of_row),
                _p(cache.tables), cache.tables.shape[1], _p(row0), _p(nrows), _p(rows), n, H, rank, Dk, float(scale),
                int(window or 0), sink, splits, _p(acc), _p(ml), _p(err), _stream()), "latent_attention_mma")
        if plan.n_portions:
            row0, nrows, n = plan.tiles(LATENT_TILE_ROWS)
            launch(row0, nrows, None, n)
        if plan.n_decode:
            # single tokens: few groups (one per token and 16 heads), so a group's key tiles are dealt to several
            # CTAs where that fills more of the GPU, and a second launch merges what they leave
            keys = plan.max_len if not window else min(plan.max_len, int(window) + 1)
            tiles = -(-keys // 64) + 1
            cells = plan.n_decode * -(-H // 16)
            splits = max(1, min(tiles, 2 * sm_count() // max(1, cells), 16))
            if splits > 1:
                acc = torch.empty(cells * splits * 16 * rank, dtype=torch.float32, device=out.device)
                ml = torch.empty(cells * splits * 16 * 2, dtype=torch.float32, device=out.device)
                launch(None, None, plan.decode_rows, plan.n_decode, splits, acc, ml)
            else:
                launch(None, None, plan.decode_rows, plan.n_decode)
        return
    library.check(library.load().cuca_latent_attention_s(
        _p(qk), _p(out), _p(pool), dtype_code(pool.dtype), pool.shape[0], pool.shape[2], _p(step.positions),
        _p(step.seq_of_row), _p(cache.tables), cache.tables.shape[1], qk.shape[0], H, rank, Dk, float(scale),
        int(window or 0), sink, _p(err), _stream()), "latent_attention")


# ------------------------------------------------------------------ attention whose values are wider or narrower than its keys
def rope_store_general(qkv, k_col, v_col, positions, seq_of_row, tables, cos, sin, rotary_dim, adjacent, kpool, vpool,
                       block_size, n_heads, n_kv_heads, head_dim, v_head_dim, err, v_split: int = 1,
                       v_row_dim: int = 0) -> None:
    """Rotate the first `rotary_dim` values of every q head (in place) and k head of `qkv` rows (q heads at column 0,
    k heads at `k_col`, v heads of `v_head_dim` at `v_col`), pairs (i, i + n/2) or, `adjacent`, (2i, 2i + 1); write
    k and v to the row's page. `v_split` r > 1: the value pool's memory is r slabs of heads r times narrower.
    `v_row_dim` n > 0: a row's value heads hold n values and the pool's `v_head_dim` >= n; the rest is kept as zeros."""
    _cuda(qkv, positions, seq_of_row, kpool, vpool)
    library.check(library.load().cuca_rope_store_general(
        _p(qkv), dtype_code(qkv.dtype), qkv.stride(0), int(k_col), int(v_col), _p(positions), _p(seq_of_row),
        _p(tables), tables.shape[1], _p(cos), _p(sin), cos.shape[0] if cos is not None else 0, int(rotary_dim),
        int(bool(adjacent)), _p(kpool), _p(vpool), kpool.shape[0], int(block_size), qkv.shape[0], n_heads, n_kv_heads,
        head_dim, v_head_dim, int(v_split), int(v_row_dim), _p(err), _stream()), "rope_store_general")


def attention_generic_v(q, q_stride, out, kpool, vpool, positions, seq_of_row, tables, n_heads, n_kv_heads,
                        head_dim, v_head_dim, scale, window, err, **options) -> None:
    """The plain attention kernel with value heads of their own size (`vpool`: [pages, kv heads, block, v_head_dim]);
    `options`: see `attention_options`."""
    _cuda(q, out, kpool, vpool)
    opt = attention_options(n_heads, scale, window, gate_width=n_heads * v_head_dim, **options)
    library.check(library.load().cuca_attention_generic_o(
        _p(q), int(q_stride), _p(out), out.stride(0), dtype_code(out.dtype), _p(kpool), _p(vpool), kpool.shape[0],
        kpool.shape[2], _p(positions), _p(seq_of_row), _p(tables), tables.shape[1], out.shape[0], n_heads,
        n_kv_heads, head_dim, v_head_dim, ctypes.addressof(opt), _p(err), _stream()), "attention_generic")


def norm_rope_store(qkv, k_col, v_col, positions, seq_of_row, tables, cos, sin, rotary_dim, adjacent, q_norm, k_norm,
                    v_norm: bool, eps: float, kpool, vpool, block_size, n_heads, n_kv_heads, head_dim, v_head_dim, err,
                    v_split: int = 1, q_out=None, v_row_dim: int = 0, whole: bool = False, q_temp=None,
                    unit: bool = False, q_mul=None, key_scale=None) -> None:
    """`rope_store_general` with norms per head in 32-bit before the rotation: q / rms(q) * q_norm, k likewise with
    k_norm (None: no norm), and with `v_norm` v / rms(v) before it is kept. q is rewritten in place, or goes to
    `q_out` [rows, heads * head_dim] of the pools' dtype (32-bit rows beside 16-bit pools). `v_row_dim` n > 0: a row's
    value heads hold n values (the norm is over those) and the pool's `v_head_dim` >= n; the rest is kept as zeros.
    `whole`: the norm of q (and of k) is over the whole projection, all heads at once, with weights [heads * head_dim].
    `q_temp` (coef, every): the query at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1).
    `unit`: the norms per head have no weight. `q_mul` (32-bit, one per query head): a factor on the head's queries, after
    the norm. `v_col` may be `k_col`: the values are then the keys as projected. `key_scale` (with `unit`, without rotation;
    `vpool` None): the page rows hold the keys as projected and `key_scale` the factors their norms would have been."""
    _cuda(qkv, positions, seq_of_row, kpool, vpool, q_norm, k_norm, q_out)
    coef, every = (float(q_temp[0]), int(q_temp[1])) if q_temp else (0.0, 0)
    library.check(library.load().cuca_norm_rope_store_u(
        _p(qkv), dtype_code(qkv.dtype), qkv.stride(0), int(k_col), int(v_col), _p(q_out), dtype_code(kpool.dtype),
        _p(positions), _p(seq_of_row), _p(tables), tables.shape[1], _p(cos), _p(sin),
        cos.shape[0] if cos is not None else 0, int(rotary_dim), int(bool(adjacent)), _p(q_norm), _p(k_norm),
        int(bool(v_norm)), float(eps), _p(kpool), _p(vpool), kpool.shape[0], int(block_size), qkv.shape[0], n_heads,
        n_kv_heads, head_dim, v_head_dim, int(v_split), int(v_row_dim), int(bool(whole)), coef, every, int(bool(unit)),
        _per_head(q_mul, n_heads, "factors on the queries"), _key_scale(key_scale), _p(err), _stream()),
        "norm_rope_store")


def sigmoid_gate_(a, gate) -> None:
    """a *= sigmoid(gate); both [rows, n] of one dtype, rows of any stride."""
    _cuda(a, gate)
    library.check(library.load().cuca_sigmoid_gate(_p(a), a.stride(0), _p(gate), gate.stride(0), dtype_code(a.dtype),
                                                   a.shape[0], a.shape[1], _stream()), "sigmoid_gate")


def gate_merge(parts, gate, out, n_heads, v_head_dim) -> None:
    """out[r, h] = [parts[0][r, h] | parts[1][r, h] | ...] * sigmoid(gate[r, h]) (gate None: no gate); parts:
    [split, rows, heads * v_head_dim / split] contiguous."""
    _cuda(parts, gate, out)
    library.check(library.load().cuca_gate_merge(_p(parts), _p(gate), gate.stride(0) if gate is not None else 0, _p(out),
                                                 dtype_code(out.dtype), out.shape[0], n_heads, v_head_dim,
                                                 parts.shape[0], _stream()), "gate_merge")


# ------------------------------------------------------------------ several copies of the residual stream
STREAMS_MAX = 16  # `cuca_streams_max` says the same


def spread_streams(x, X, copies: int) -> None:
    """X[r, s] = x[r] for every copy s; x: [rows, E], X: [rows, copies * E], both 32-bit."""
    _cuda(x, X)
    library.check(library.load().cuca_spread_streams(_p(x), _p(X), x.shape[0], int(copies), x.shape[1], _stream()),
                  "spread_streams")


def streams_read(X, read, weight, out, copies: int, eps: float, rows=None) -> None:
    """out = RMSNorm(sum_s read[s] X[:, s]) * weight (read None: the plain sum); `rows` gathers rows of X."""
    _cuda(X, read, weight, out, rows)
    library.check(library.load().cuca_streams_read(_p(X), _p(read), _p(weight), _p(out), dtype_code(out.dtype),
                                                   _p(rows), out.shape[0], int(copies), out.shape[1], float(eps),
                                                   _stream()), "streams_read")


def streams_write(X, y, mix, write, copies: int, eps: float, read2=None, weight2=None, out2=None) -> None:
    """X[:, t] <- sum_s mix[s, t] X[:, s] + write[t] y, all copies from the old ones; with `out2` also
    out2 = RMSNorm(sum_t read2[t] X[:, t]) * weight2 of the new copies."""
    _cuda(X, y, mix, write, read2, weight2, out2)
    library.check(library.load().cuca_streams_write(
        _p(X), _p(y), _p(mix), _p(write), _p(read2), _p(weight2), _p(out2),
        dtype_code(out2.dtype) if out2 is not None else 0, y.shape[0], int(copies), y.shape[1], float(eps), _stream()),
        "streams_write")


def pair_norm_add(x, a, b, wa, wb, c: float, eps: float, store: bool = False) -> None:
    """x += c (RMSNorm(a) * wa + RMSNorm(b) * wb), or x = ... with `store`; all 32-bit [rows, E]."""
    _cuda(x, a, b, wa, wb)
    library.check(library.load().cuca_pair_norm_add(_p(x), _p(a), _p(b), _p(wa), _p(wb), float(c), int(bool(store)),
                                                    x.shape[0], x.shape[1], float(eps), _stream()), "pair_norm_add")


# ------------------------------------------------------------------ mixers with a matrix state per head
MATRIX_STATE_MAX_DIM = 1024  # `cuca_matrix_state_max_dim` says the same


def delta_scan(qkv, a_raw, dt_bias, a_log, b_src, b_col, state, out, step, H, G, d, dv) -> None:
    """The delta rule with a decay per key channel along every request's rows (see `parts/recurrent.py:GatedDelta`).
    `qkv`, `a_raw` and column `b_col`.. of `b_src` hold pre-activations and are rewritten in place (unit vectors,
    decays, the write gate) before the scan; two launches."""
    _cuda(qkv, a_raw, dt_bias, a_log, b_src, state, out)
    library.check(library.load().cuca_delta_scan(
        _p(qkv), qkv.stride(0), _p(a_raw), a_raw.stride(0), _p(dt_bias), _p(a_log), _p(b_src), b_src.stride(0), int(b_col),
        _p(state),
        _p(out), _p(step.seq_of_row), _p(step.req_row0), _p(step.req_count), _p(step.slots), qkv.shape[0], step.n_seqs,
        H, G, d, dv, _stream()), "delta_scan")
    library.launches += 1


def mlstm_scan(proj, q_col, k_col, v_col, i_col, f_col, i_bias, f_bias, cap, mem, nrm, mx, out, step, H, d, dv) -> None:
    _cuda(proj, mem, nrm, mx, out)
    # the new normaliser and running maximum of every (request, head), set aside until every block has read the old
    aside = torch.empty(step.n_seqs * H * (d + 1), dtype=torch.float32, device=out.device)
    library.check(library.load().cuca_mlstm_scan(
        _p(proj), proj.stride(0), int(q_col), int(k_col), int(v_col), int(i_col), int(f_col), _p(i_bias), _p(f_bias),
        float(cap), _p(mem), _p(nrm), _p(mx), _p(out), _p(aside), _p(step.req_row0), _p(step.req_count), _p(step.slots),
        proj.shape[0], step.n_seqs, H, d, dv, _stream()), "mlstm_scan")
    library.launches += 2  # the gates are prepared by a launch of their own, the new n and m moved in by another


def forget_scan(proj, q_col, f_col, v_col, f_bias, lower, state, out, step, H, d, dv) -> None:
    """Linear attention whose forget gate is also one minus its write strength, along every request's rows (see
    `parts/recurrent.py:ForgetGateAttention`). The q and gate columns of `proj` hold pre-activations and are rewritten
    in place (silu; the gate above its lower bound) before the scan; two launches."""
    _cuda(proj, f_bias, lower, state, out)
    library.check(library.load().cuca_forget_scan(
        _p(proj), proj.stride(0), int(q_col), int(f_col), int(v_col), _p(f_bias), _p(lower), _p(state), _p(out),
        _p(step.seq_of_row), _p(step.req_row0), _p(step.req_count), _p(step.slots), proj.shape[0], step.n_seqs, H, d, dv,
        _stream()), "forget_scan")
    library.launches += 1


def retention_scan(proj, q_col, k_col, v_col, decay, cos, sin, rot_dims, k_scale, state, out, step, H, d, dv, err) -> None:
    """Retention along every request's rows: S <- decay[h] S + k v^T, o = S^T q per head (see
    `parts/recurrent.py:Retention`). The q and k columns of the 32-bit `proj` are rewritten in place before the scan
    (the first `rot_dims` values of a head turned by the row's position in pairs (i, i + rot_dims / 2), k times
    `k_scale`); two launches."""
    _cuda(proj, decay, state, out, cos, sin)
    library.check(library.load().cuca_retention_scan(
        _p(proj), proj.stride(0), int(q_col), int(k_col), int(v_col), _p(decay), _p(cos), _p(sin),
        cos.shape[0] if cos is not None else 0, int(rot_dims), float(k_scale), _p(step.positions), _p(state), _p(out),
        _p(step.seq_of_row), _p(step.req_row0), _p(step.req_count), _p(step.slots), proj.shape[0], step.n_seqs, H, d, dv,
        _p(err), _stream()), "retention_scan")
    library.launches += 1


def lightning_scan(proj, decay, state, out, step, H, d, dv) -> None:
    """Lightning attention along every request's rows: the recurrence of retention on silu(q), silu(k), silu(v) (see
    `parts/recurrent.py:Lightning`). The first H (2 d + dv) columns of the 32-bit `proj` hold q, k, v before their
    activation and may be rewritten in place; two launches, or one where every request brings a single token."""
    _cuda(proj, decay, state, out)
    if step.all_single():
        library.check(library.load().cuca_lightning_step(
            _p(proj), proj.stride(0), 0, _p(decay), _p(state), _p(out), _p(step.req_row0), _p(step.req_count),
            _p(step.slots), step.n_seqs, H, d, dv, _stream()), "lightning_step")
        return
    library.check(library.load().cuca_lightning_scan(
        _p(proj), proj.stride(0), 0, _p(decay), _p(state), _p(out), _p(step.seq_of_row), _p(step.req_row0),
        _p(step.req_count), _p(step.slots), proj.shape[0], step.n_seqs, H, d, dv, _stream()), "lightning_scan")
    library.launches += 1


def row_norm_gate(o, weight, gate, out, eps: float) -> None:
    """out[r] = o[r] / rms(o[r]) * weight * sigmoid(gate[r]) over whole rows; gate: rows of any stride."""
    _cuda(o, weight, gate, out)
    library.check(library.load().cuca_row_norm_gate(_p(o), _p(weight), _p(gate), dtype_code(gate.dtype), gate.stride(0),
                                                    _p(out), dtype_code(out.dtype), o.shape[0], o.shape[1], float(eps),
                                                    _stream()), "row_norm_gate")


LIGHTNING_CHUNK, LIGHTNING_CHUNK_MAX_DIM = 64, 256  # `cuca_lightning_chunk_tokens` / `_max_dim` say the same
LIGHTNING_CHUNKED_FROM = 32  # steps with a portion at least this long, in the serving precision only


def lightning_chunks(step, dtype, d: int) -> int:
    """Chunks of this step's portions if it should run chunk by chunk on the tensor cores, else 0 (token by token: single
    tokens, short portions, the 32-bit path always)."""
    counts = step.host.get("counts") if step.static_max_len is None else None
    if dtype != torch.bfloat16 or d > LIGHTNING_CHUNK_MAX_DIM or not counts or max(counts) < LIGHTNING_CHUNKED_FROM:
        return 0
    return sum(-(-c // LIGHTNING_CHUNK) for c in counts)


def lightning_chunked(proj, decay, state, out, step, n_chunks: int, H, d, dv) -> None:
    """`lightning_scan` chunk by chunk from a bfloat16 `proj` (read only); three launches."""
    _cuda(proj, decay, state, out)
    if proj.dtype != torch.bfloat16:
        raise library.KernelError("lightning_chunked takes a bfloat16 projection")
    chunks = torch.empty(n_chunks, H, dv, d, dtype=torch.float32, device=out.device)
    library.check(library.load().cuca_lightning_chunked(
        _p(proj), proj.stride(0), 0, _p(decay), _p(state), _p(chunks), _p(out), _p(step.req_row0), _p(step.req_count),
        _p(step.slots), step.n_seqs, n_chunks, H, d, dv, _stream()), "lightning_chunked")
    library.launches += 2


def head_norm_gate(o, weight, per_head: bool, gate, out, H, dv, eps, gate_act: str = "sigmoid") -> None:
    """out[r, h] = o[r, h] / rms(o[r, h]) * weight * act(gate[r, h]); weight [dv] for every head or [H dv], or None;
    act the sigmoid or, `gate_act` "silu", g sigmoid(g)."""
    _cuda(o, weight, gate, out)
    library.check(library.load().cuca_head_norm_gate_act(
        _p(o), _p(weight), dv if per_head else 0, _p(gate), dtype_code(gate.dtype) if gate is not None else 0,
        gate.stride(0) if gate is not None else 0, 1 if gate_act == "silu" else 0, _p(out), dtype_code(out.dtype),
        o.shape[0], H, dv, float(eps), _stream()), "head_norm_gate")


# ------------------------------------------------------------------ routed feed-forward
MOE_MAX_EXPERTS, MOE_MAX_TOP = 1024, 32


def moe_route(logits, top, idx, wts, dense=None) -> None:
    _cuda(logits, idx, wts, dense)
    library.check(library.load().cuca_moe_route(_p(logits), logits.shape[0], logits.shape[1], int(top), _p(idx),
                                                _p(wts), _p(dense), _stream()), "moe_route")


def moe_act_dense(u, dense, a, E, F) -> None:
    _cuda(u, dense, a)
    library.check(library.load().cuca_moe_act_dense(_p(u), _p(dense), _p(a), dtype_code(u.dtype), u.shape[0], E, F,
                                                    _stream()), "moe_act_dense")


def moe_sparse(h, w_up, w_down, idx, wts, a, y, store, top, E, F, glu: bool = False) -> None:
    """y (+)= sum over a token's chosen experts of weight * down_e(act_e h), reading only those experts. Plain:
    act = relu(up h)^2, `w_up` [E F, K], `w_down` [N, E F]. `glu`: act = silu(gate h) * (up h), `w_up` [2 C, K] (all
    gates, then all ups), `w_down` [N, C], C >= E F. Pairs that name expert E or more (experts without weights) are
    skipped."""
    _cuda(h, w_up, w_down, idx, wts, a, y)
    library.check(library.load().cuca_moe_sparse(_p(h), _p(w_up), _p(w_down), _p(idx), _p(wts), _p(a), _p(y),
                                                 int(bool(store)), dtype_code(h.dtype), h.shape[0], int(top), E, F,
                                                 h.shape[1], y.shape[1], int(bool(glu)), w_down.shape[1], _stream()),
                  "moe_sparse")
    library.launches += 1


def moe_route_scored(logits, correction, n_real, top, idx, wts, dense=None, ident=None) -> None:
    """Scores s = softmax over all router outputs; the `top` largest of s + correction are chosen (`correction` None:
    of s); weights s / (sum of the chosen s + 1e-20). Outputs from `n_real` on are experts that return their input:
    `ident[t]` gets the sum of their chosen weights."""
    _cuda(logits, correction, idx, wts, dense, ident)
    library.check(library.load().cuca_moe_route_scored(_p(logits), _p(correction), logits.shape[0], logits.shape[1],
                                                       int(n_real), int(top), _p(idx), _p(wts), _p(dense), _p(ident),
                                                       _stream()), "moe_route_scored")


def moe_glu_dense(gu, dense, a, EF, F) -> None:
    """a[t, c] = silu(gu[t, c]) * gu[t, C + c] * w, w = dense[t, c // F] for c < EF and 1 behind (a shared expert)."""
    _cuda(gu, dense, a)
    library.check(library.load().cuca_moe_glu_dense(_p(gu), _p(dense), dense.shape[1], _p(a), dtype_code(gu.dtype),
                                                    gu.shape[0], a.shape[1], int(EF), int(F), _stream()), "moe_glu_dense")


def moe_identity_add(y, h, ident, store: bool) -> None:
    """y[t] (+)= ident[t] * h[t]."""
    _cuda(y, h, ident)
    library.check(library.load().cuca_moe_identity_add(_p(y), _p(h), dtype_code(h.dtype), _p(ident), int(bool(store)),
                                                       h.shape[0], h.shape[1], _stream()), "moe_identity_add")


def moe_route_grouped(logits, experts: int, groups: int, keep: int, top: int, scale: float, shared: bool, idx, wts,
                      dense=None) -> None:
    """Scores sigmoid(logits); of `groups` equal groups of neighbouring experts the `keep` with the largest sums of their
    two largest scores are open, the `top` largest scores among those are chosen, weights score * scale. `shared`: the
    logits' last column is a shared expert's; it becomes the last entry (number `experts`) with weight sigmoid."""
    _cuda(logits, idx, wts, dense)
    library.check(library.load().cuca_moe_route_grouped(
        _p(logits), logits.shape[0], int(experts), int(groups), int(keep), int(top), float(scale), int(bool(shared)),
        _p(idx), _p(wts), _p(dense), _stream()), "moe_route_grouped")


MOE_ROUTER_MAX_OUTPUTS = 64


def moe_router_grouped(h, w, experts: int, groups: int, keep: int, top: int, scale: float, shared: bool, idx, wts) -> None:
    """`moe_route_grouped` from the activations h and the router's rows w (up to `MOE_ROUTER_MAX_OUTPUTS`), one launch."""
    _cuda(h, w, idx, wts)
    library.check(library.load().cuca_moe_router_grouped(
        _p(h), _p(w), dtype_code(h.dtype), h.shape[0], h.shape[1], int(experts), int(groups), int(keep), int(top),
        float(scale), int(bool(shared)), _p(idx), _p(wts), _stream()), "moe_router_grouped")


def moe_sparse_capped(h, w_gu, w_down, idx, wts, a, y, store, E: int, F: int, Fs: int, limit: float, limit_s: float,
                      alpha: float) -> None:
    """`moe_sparse` for experts that are capped gated units (`glu_capped`): `w_gu` [2 C, K] all gates then all ups,
    `w_down` [N, C], C = E F + Fs. Entry number E is the shared expert of Fs rows with cap `limit_s`."""
    _cuda(h, w_gu, w_down, idx, wts, a, y)
    library.check(library.load().cuca_moe_sparse_act(
        _p(h), _p(w_gu), _p(w_down), _p(idx), _p(wts), _p(a), a.stride(0), _p(y), int(bool(store)), dtype_code(h.dtype),
        h.shape[0], idx.shape[1], E, F, Fs, h.shape[1], y.shape[1], 2, w_down.shape[1], float(limit), float(limit_s),
        float(alpha), _stream()), "moe_sparse")
    library.launches += 1


def moe_glu_capped_dense(gu, dense, a, EF: int, F: int, limit: float, limit_s: float, alpha: float) -> None:
    """a[t, c] = capped unit of (gu[t, c], gu[t, C + c]) * w: c < EF: w = dense[t, c // F] and cap `limit`; behind (a
    shared expert): w = dense[t, EF // F] and cap `limit_s`."""
    _cuda(gu, dense, a)
    library.check(library.load().cuca_moe_glu_capped_dense(
        _p(gu), _p(dense), dense.shape[1], _p(a), dtype_code(gu.dtype), gu.shape[0], a.shape[1], int(EF), int(F),
        float(limit), float(limit_s), float(alpha), _stream()), "moe_glu_capped_dense")


# ------------------------------------------------------------------ a sublayer's output on its way to the stream
MAX_TERMS = 8  # `cuca_max_terms` says the same


class _Terms(ctypes.Structure):
    """The kernels' description of a weighted sum of terms (`csrc/sublayer_output.cu:CucaTerms`)."""

    _fields_ = [("n", ctypes.c_int), ("data", ctypes.c_void_p * MAX_TERMS), ("slices", ctypes.c_int * MAX_TERMS),
                ("stride", ctypes.c_size_t * MAX_TERMS), ("scale", ctypes.c_float * MAX_TERMS)]


def _terms(terms) -> _Terms:
    """`terms`: (32-bit tensor [rows, E] or `PartialSums`, factor) pairs."""
    t = _Terms()
    if len(terms) > MAX_TERMS:
        raise library.KernelError(f"{len(terms)} terms exceed {MAX_TERMS}")
    t.n = len(terms)
    for i, (x, scale) in enumerate(terms):
        if isinstance(x, PartialSums):
            t.data[i], t.slices[i], t.stride[i] = x.data.data_ptr(), x.slices, x.slice_stride
        else:
            if x.dtype != torch.float32 or not x.is_contiguous():
                raise library.KernelError("a term is a contiguous 32-bit tensor or a contraction's K slices")
            t.data[i], t.slices[i], t.stride[i] = x.data_ptr(), 1, 0
        t.scale[i] = float(scale)
    return t


def norm_add(x, terms, weight, eps: float, out=None, center: bool = True) -> None:
    """x += N(y) * weight with y the weighted sum of `terms`; `out` (or None) = the new x in out's dtype. N is the
    layer norm, or the RMS norm with `center` False."""
    _cuda(x, weight, out)
    t = _terms(terms)
    library.check(library.load().cuca_norm_add(_p(x), ctypes.addressof(t), _p(weight), _p(out),
                                               dtype_code(out.dtype) if out is not None else 0, x.shape[0], x.shape[1],
                                               float(eps), int(bool(center)), _stream()), "norm_add")


def layer_norm(x, weight, out, eps: float, rows=None) -> None:
    """out[r] = (x - mean) / sqrt(mean((x - mean)^2) + eps) * weight of row r (or rows[r]) of x."""
    _cuda(x, weight, out, rows)
    library.check(library.load().cuca_layer_norm(_p(x), _p(weight), _p(out), dtype_code(out.dtype), _p(rows), out.shape[0],
                                                 x.shape[1], float(eps), _stream()), "layer_norm")


def add_terms(x, terms, store: bool) -> None:
    """x (+)= the weighted sum of `terms`."""
    _cuda(x)
    t = _terms(terms)
    library.check(library.load().cuca_add_terms(_p(x), ctypes.addressof(t), int(bool(store)), x.numel(), _stream()),
                  "add_terms")


def round_rows(x, out) -> None:
    """out = x in out's dtype."""
    _cuda(x, out)
    library.check(library.load().cuca_round_rows(_p(x), _p(out), dtype_code(out.dtype), x.numel(), _stream()),
                  "round_rows")


# ------------------------------------------------------------------ blocks that norm the sum
def sum_norm(x, terms, scale, weight, alpha: float, eps: float, out=None) -> None:
    """x <- N(alpha x + scale * y) * weight in place with y the weighted sum of `terms` and N the RMS norm; `out` (or None)
    = the new x in out's dtype. `scale`: a factor per channel, or None."""
    _cuda(x, scale, weight, out)
    t = _terms(terms)
    library.check(library.load().cuca_sum_norm(_p(x), ctypes.addressof(t), _p(scale), _p(weight), float(alpha), float(eps),
                                               _p(out), dtype_code(out.dtype) if out is not None else 0, x.shape[0],
                                               x.shape[1], _stream()), "sum_norm")


def sum_norm_shift_supported(width: int) -> bool:
    return bool(library.load().cuca_sum_norm_shift_supported(int(width)))


def sum_norm_shift(x, terms, scale, weight, alpha: float, eps: float, x_out, mix, kept, out, step) -> None:
    """`sum_norm` out of place, and out[r] = x_out[r] + (x_out[r-1] - x_out[r]) * mix of the new rows; the row before a
    request's first row of the step is `kept[slot]`, which then becomes the request's last row."""
    _cuda(x, scale, weight, x_out, mix, kept, out)
    t = _terms(terms)
    library.check(library.load().cuca_sum_norm_shift(
        _p(x), ctypes.addressof(t), _p(scale), _p(weight), float(alpha), float(eps), _p(x_out), _p(mix), _p(kept), _p(out),
        dtype_code(out.dtype), _p(step.seq_of_row), _p(step.req_row0), _p(step.req_count), x.shape[0], step.n_seqs,
        x.shape[1], _stream()), "sum_norm_shift")


def shift_rows(x, mix, kept, out, step) -> None:
    """out[r] = x[r] + (x[r-1] - x[r]) * mix; the kept rows as in `sum_norm_shift`."""
    _cuda(x, mix, kept, out)
    library.check(library.load().cuca_shift_rows(_p(x), _p(mix), _p(kept), _p(out), dtype_code(out.dtype),
                                                 _p(step.seq_of_row), _p(step.req_row0), _p(step.req_count), _p(step.slots),
                                                 x.shape[0], step.n_seqs, x.shape[1], _stream()), "shift_rows")
