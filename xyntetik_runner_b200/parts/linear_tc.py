"""The tensor-core route of ``Linear``: bfloat16 activations times a bfloat16 matrix on tcgen05."""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels

ENABLED = True         # (False sends every product to the float32 FMA kernel: a test may set it to bisect a difference)


class Pending:
    """A product whose sum over its K slices is still to be taken: float32 partial sums [splits][n][width] in a
    slab of the product's workspace, to be summed into `out` (plus the bias).  Whoever takes the sum -- ``finish``,
    or a kernel that does it in passing -- calls ``release`` afterwards; until then the slab is this product's
    alone, so a part may start another product before it finishes this one."""

    def __init__(self, sums: "kernels.PartialSums", bias: Optional[torch.Tensor], out: torch.Tensor, accumulate: bool):
        self.sums, self.partial, self.splits = sums, sums.partial, sums.splits
        self.bias, self.out, self.accumulate = bias, out, accumulate

    def release(self) -> None:
        self.sums.release()

    def finish(self) -> None:
        kernels.finish_plain(self.partial, self.splits, self.bias, self.out, self.accumulate)
        self.release()

    def finish_norm(self, x, w, out, eps, w2=None, out2=None) -> None:
        """The sum added into x and the norm of the new rows into `out` (and with `w2` into `out2`), in one pass."""
        kernels.finish_add_rmsnorm(self.partial, self.splits, self.bias, x, w, out, eps, w2, out2)
        self.release()

    def join(self, later: "Pending") -> Optional["Pending"]:
        """One pending sum for this product's and a later one's, when both add into the same rows, their slabs lie one right
        behind the other and at most one has a bias: the partial sums then read as one array [splits + later.splits][n][width],
        summed in that order by one kernel.  (Side-by-side sublayers that add into the stream one after the other leave such a
        pair.)  None when they do not join."""
        if not (isinstance(later, Pending) and self.accumulate and later.accumulate and self.out.data_ptr() == later.out.data_ptr()
                and self.out.shape == later.out.shape and (self.bias is None or later.bias is None)):
            return None
        if later.partial.data_ptr() != self.partial.data_ptr() + 4 * self.partial.numel():
            return None
        return _Joined(self, later)


class _Joined(Pending):
    def __init__(self, first: Pending, second: Pending):
        ws = first.sums._ws
        at = (first.partial.data_ptr() - ws.scratch.data_ptr()) // 4
        self.parts = (first, second)
        self.partial = ws.scratch[at:at + first.partial.numel() + second.partial.numel()]
        self.splits = first.splits + second.splits
        self.bias = first.bias if first.bias is not None else second.bias
        self.out, self.accumulate = first.out, True

    def release(self) -> None:
        for p in self.parts:
            p.release()


def usable(lin, x, out, accumulate) -> bool:
    return ENABLED and lin.weight is not None and kernels.gemm_tc_supported(x, lin.weight, out)


def run(lin, x, out, accumulate, defer=False, act=kernels.ACT_NONE, alpha=1.0):
    epi = kernels.EPI_ADD if accumulate else kernels.EPI_STORE
    w, packed_rows = (lin.packed, lin.n_out) if lin.packed is not None else (lin.weight, None)
    if defer:
        assert act == kernels.ACT_NONE
        sums = kernels.gemm_tc_deferred(x, w, out, lin.bias, epi, packed_rows=packed_rows, alpha=alpha)
        if sums is None:
            return None
        return Pending(sums, lin.bias, out, accumulate)
    kernels.gemm_tc(x, w, out, lin.bias, epi, packed_rows=packed_rows, act=act, alpha=alpha)
    return None
