"""What every part needs of its surroundings: device, compute dtype, the error word, projections."""
from __future__ import annotations

import torch

from .kernels import library, ops


class DeviceFault(RuntimeError):
    """A kernel recorded a bad index (token id, page id) or a wait that ran out."""


_ERR_TEXT = {
    1: "a token id or position outside its table reached a kernel",
    2: "a page id outside the pool, or a position without a page, reached a kernel",
    3: "a bounded wait inside a kernel ran out",
    4: "a kernel found its shared memory laid out otherwise than its budget assumes",
}


class Runtime:
    """Device, compute dtype (float32: true 32-bit everywhere; bfloat16: serving precision) and shared helpers."""

    def __init__(self, device="cuda:0", dtype: torch.dtype = torch.bfloat16):
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"compute dtype must be float32 or bfloat16, not {dtype}")
        self.device = torch.device(device)
        self.dtype = dtype
        if self.device.type != "cuda":
            raise library.KernelLibraryError(
                "cuca_b200 runs on a CUDA device only: there is no CPU path (device given: %s)" % device)
        if not torch.cuda.is_available():
            raise library.KernelLibraryError("no CUDA device is visible: cuca_b200 has no CPU path")
        library.load()
        torch.cuda.set_device(self.device)
        self.err = torch.zeros(1, dtype=torch.int32, device=self.device)
        self.use_partials = True  # few-token contractions may leave their K slices unadded for the next reader

    # ---------------------------------------------------------------- helpers
    def empty(self, *shape, dtype=None) -> torch.Tensor:
        return torch.empty(*shape, dtype=dtype or self.dtype, device=self.device)

    def linear(self, a, w, out=None, epilogue=ops.EPI_STORE, bias=None, out_dtype=None):
        """out = epilogue(a @ w.T): store, add to the 32-bit stream, or SwiGLU over stacked [gate; up]."""
        n = w.shape[0] // 2 if epilogue == ops.EPI_SWIGLU else w.shape[0]
        if out is None:
            out = self.empty(a.shape[0], n, dtype=out_dtype or self.dtype)
        ops.gemm(a, w, out, epilogue, bias, self.err)
        return out

    def stream(self, x) -> "ResidualStream":
        """`x` as a residual stream: itself if it is one already, else a 32-bit tensor wrapped."""
        return x if isinstance(x, ResidualStream) else ResidualStream(self, x)

    def check_device_errors(self) -> None:
        """Read the error word (synchronises); raise if a kernel recorded a fault."""
        code = int(self.err.item())
        if code:
            self.raise_device_error(code)

    def raise_device_error(self, code: int) -> None:
        """A kernel recorded `code` (read by the caller, e.g. along with a step's sampled tokens): clear the
        word and raise."""
        self.err.zero_()
        raise DeviceFault(_ERR_TEXT.get(code, f"device error {code}"))


class ResidualStream:
    """The 32-bit residual stream of a step, `[rows, width]`, as blocks and parts get it.

    Over few tokens (up to a few hundred: the kernel library says how many) a contraction into the stream is cut
    along K over the SMs and leaves its slices unadded (`add_linear`); whoever reads the stream next adds them. That hand-over is this object's business, not the
    parts': `data` adds pending slices before it returns the tensor, so a part written against `data` (read it,
    update it in place) is always right. A reader that can add the slices while it reads, in the same pass over
    memory (the RMSNorm kernel), asks for `take()` instead and gets the tensor and the slices."""

    def __init__(self, runtime: Runtime, tensor: torch.Tensor):
        if tensor.dtype != torch.float32:
            raise ValueError("the residual stream is 32-bit in every mode")
        self.rt = runtime
        self._tensor = tensor
        self._pending = None
        self._unwritten = False
        self._rounded = None  # the stream in the compute dtype, while nothing has touched the stream since it was made
        self._unsummed = None  # (output, norm, alpha, scale) of `defer_sum_norm`: the stream is what that makes of it

    @classmethod
    def unwritten(cls, runtime: "Runtime", rows: int, width: int) -> "ResidualStream":
        """A stream that holds nothing yet (a sublayer's output gathered apart from the model's stream, for a norm
        on it): the first contraction added to it is stored instead, so it needs no zeroing."""
        s = cls(runtime, torch.empty(rows, width, dtype=torch.float32, device=runtime.device))
        s._unwritten = True
        return s

    def replace(self, tensor: torch.Tensor) -> None:
        """The stream is `tensor` from now on (an operation that rewrote the whole stream out of place)."""
        if tensor.dtype != torch.float32 or tensor.shape != self._tensor.shape:
            raise ValueError("a residual stream is replaced by a 32-bit tensor of its own shape")
        self._pending = self._rounded = self._unsummed = None
        self._tensor = tensor

    @property
    def shape(self):
        return self._tensor.shape

    @property
    def data(self) -> torch.Tensor:
        """The stream's tensor with everything added; it may be read and updated in place."""
        if self._unsummed is not None:
            self._sum_norm(*self._take_unsummed())
        self._rounded = None
        if self._unwritten:
            self._tensor.zero_()
            self._unwritten = False
        if self._pending is not None:
            ps, self._pending = self._pending, None
            ops.add_partials(self._tensor, ps)
        return self._tensor

    def take(self):
        """(tensor, pending slices or None) for a reader that adds the slices itself, in the stream too: after
        the reader's kernel the tensor must hold the sum."""
        if self._unsummed is not None:
            return self.data, None
        self._rounded = None
        if self._unwritten:
            self._tensor.zero_()
            self._unwritten = False
        ps, self._pending = self._pending, None
        return self._tensor, ps

    def claim(self):
        """(tensor, fresh) for a kernel that adds into the stream itself: `fresh` says that the stream holds nothing
        yet, so the kernel must store instead of add (nothing is zeroed for it)."""
        if self._unwritten:
            self._unwritten = False
            return self._tensor, True
        return self.data, False

    def add_linear(self, a, w, bias=None) -> None:
        """stream += a @ w.T (+ bias). Over few tokens the slices may stay pending until the next reader."""
        rt = self.rt
        self._rounded = None
        if self._unwritten:
            self._unwritten = False
            ops.gemm(a, w, self._tensor, ops.EPI_STORE, bias, rt.err)
            return
        if rt.use_partials and bias is None and ops.gemm_partial_supported(a, w):
            x = self.data  # slices of an earlier contraction go in first
            self._pending = ops.gemm_partial(a, w, rt.err)
            assert x is self._tensor
        else:
            ops.gemm(a, w, self.data, ops.EPI_RESIDUAL, bias, rt.err)

    def add(self, delta: torch.Tensor) -> None:
        """stream += delta (any float dtype, same shape)."""
        self.data.add_(delta)

    def drop_pending(self) -> None:
        """Forget unadded slices: the stream will not be read again (no logits are wanted)."""
        self._pending = self._unsummed = None

    # ------------------------------------------------ arrangements whose sublayers read the stream as it is
    def rounded(self) -> torch.Tensor:
        """The stream in the compute dtype, to be read only: what `add_normed` left, else made now. In the 32-bit mode
        the stream itself."""
        if self._rounded is None:
            x = self.data
            if x.dtype == self.rt.dtype:
                return x
            out = self.rt.empty(*x.shape)
            ops.round_rows(x, out)
            self._rounded = out
        return self._rounded

    def add_normed(self, output: "SublayerOutput", norm) -> None:
        """stream += norm(output), `norm` a part with `add_normed`; the rounded copy for the next sublayer's reader
        comes from the same pass."""
        x = self.data
        out = None if x.dtype == self.rt.dtype else self.rt.empty(*x.shape)
        norm.add_normed(x, output.terms, out)
        self._rounded = out

    # ------------------------------------------------ arrangements that norm the sum of stream and output
    def sum_normed(self, output: "SublayerOutput", norm, alpha: float, scale) -> None:
        """stream <- norm(alpha stream + scale * output), `norm` a part with `sum_norm`, `scale` a factor per channel (or
        None); the rounded copy for the next sublayer's reader comes from the same pass."""
        self.data
        self._sum_norm(output, norm, alpha, scale)

    def defer_sum_norm(self, output: "SublayerOutput", norm, alpha: float, scale) -> None:
        """`sum_normed`, left to whoever reads the stream next: a reader that mixes rows (`shifted`) does it in its own
        pass."""
        self.data
        self._rounded = None
        self._unsummed = (output, norm, alpha, scale)

    def _take_unsummed(self):
        d, self._unsummed = self._unsummed, None
        return d

    def _sum_norm(self, output, norm, alpha, scale) -> None:
        x = self._tensor
        out = None if x.dtype == self.rt.dtype else self.rt.empty(*x.shape)
        norm.sum_norm(x, output.terms, alpha, scale, out)
        self._rounded = out

    def shifted(self, mix, kept, step) -> torch.Tensor:
        """Every row mixed with its request's row before it, x[r] + (x[r-1] - x[r]) * mix, in the compute dtype, to be read
        only. `kept[slot]` stands for the row before a request's first row of the step, and becomes its last row."""
        h = self.rt.empty(*self.shape)
        if self._unsummed is not None and ops.sum_norm_shift_supported(self.shape[-1]):
            output, norm, alpha, scale = self._take_unsummed()
            x_out = torch.empty_like(self._tensor)
            norm.sum_norm(self._tensor, output.terms, alpha, scale, h, x_out=x_out, shift=(mix, kept, step))
            self._tensor, self._rounded = x_out, None
        else:
            ops.shift_rows(self.data, mix, kept, h, step)
        return h


class SublayerOutput(ResidualStream):
    """A sublayer's output gathered apart from the stream, for an arrangement that norms it before it is added: a
    weighted sum of terms, each a 32-bit tensor or the unadded K slices of a contraction. Nothing adds them up until
    a reader that takes terms does (`ResidualStream.add_normed`, `ops.add_terms`). A part writes to it as to a stream;
    `scaled(c)` is the same output with everything written through it multiplied by c."""

    def __init__(self, runtime: Runtime, rows: int, width: int):
        self.rt = runtime
        self._shape = (rows, width)
        self.factor = 1.0
        self.terms: list = []  # (tensor or PartialSums, factor)

    def scaled(self, factor: float) -> "SublayerOutput":
        view = SublayerOutput(self.rt, *self._shape)
        view.factor = self.factor * float(factor)
        view.terms = self.terms
        return view

    @property
    def shape(self):
        return torch.Size(self._shape)

    def claim(self):
        for t, c in self.terms:
            if isinstance(t, torch.Tensor) and c == self.factor:
                return t, False
        if len(self.terms) >= ops.MAX_TERMS:
            self._merge()
            return self.claim() if self.factor == 1.0 else self._fresh()
        return self._fresh()

    def _fresh(self):
        t = torch.empty(*self._shape, dtype=torch.float32, device=self.rt.device)
        self.terms.append((t, self.factor))
        return t, True

    def _merge(self) -> torch.Tensor:
        """One term with factor 1 in the place of all."""
        t = torch.empty(*self._shape, dtype=torch.float32, device=self.rt.device)
        ops.add_terms(t, self.terms, store=True)
        self.terms[:] = [(t, 1.0)]
        return t

    @property
    def data(self) -> torch.Tensor:
        if self.factor != 1.0:
            raise ValueError("a scaled view of a sublayer's output is only written to")
        if len(self.terms) == 1 and isinstance(self.terms[0][0], torch.Tensor) and self.terms[0][1] == 1.0:
            return self.terms[0][0]
        return self._merge()

    def take(self):
        return self.data, None

    def add_linear(self, a, w, bias=None) -> None:
        rt = self.rt
        if (rt.use_partials and bias is None and len(self.terms) < ops.MAX_TERMS - 1
                and ops.gemm_partial_supported(a, w)):
            self.terms.append((ops.gemm_partial(a, w, rt.err), self.factor))
            return
        t, fresh = self.claim()
        ops.gemm(a, w, t, ops.EPI_STORE if fresh else ops.EPI_RESIDUAL, bias, rt.err)

    def replace(self, tensor: torch.Tensor) -> None:
        raise ValueError("a sublayer's output is written to, not replaced")

    def drop_pending(self) -> None:
        pass
