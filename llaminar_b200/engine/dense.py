"""Linear layers with unquantised matrices, shared by the models with per-layer mixers (engine/stack.py, engine/mixers.py)."""
from __future__ import annotations

import torch


GROUPED_ROWS, GROUPED_SIZE = 64, 1 << 21        # batches and matrices that the small-batch kernel takes in groups of rows


def pad8(n: int) -> int:
    return -(-n // 8) * 8


def pad_to(x: torch.Tensor, *shape: int) -> torch.Tensor:
    out = torch.zeros(*shape, dtype=x.dtype, device=x.device)
    out[tuple(slice(0, n) for n in x.shape)] = x
    return out


class DenseLinear:
    """y = x W^T with W as it is stored (bf16, or float in 32-bit mode)."""

    def __init__(self, weight: torch.Tensor):
        self.w = weight.contiguous()
        self.n_out, self.k = weight.shape[0], weight.shape[1]

    def nbytes(self) -> int:
        return self.w.numel() * self.w.element_size()

    def _groups(self, x: torch.Tensor) -> int:
        """In how many groups of at most eight rows the small-batch kernel takes this product (0: it does not): one, or more for
        a small matrix, which stays in L2 between the groups."""
        from ..ops import dense as ops
        rows, n = x.shape[0], ops.GEMV_MAX_ROWS
        g = 1 if rows <= n else rows // n if rows % n == 0 and rows <= GROUPED_ROWS and self.w.numel() <= GROUPED_SIZE else 0
        return g if g and ops.gemv_fits(self.w, x[:n]) else 0

    def _gemv(self, x: torch.Tensor, out: torch.Tensor, g: int, **kw) -> None:
        from ..ops import dense as ops
        split = lambda t: t.unsqueeze(0) if g == 1 else t.unflatten(0, (g, -1))
        ops.gemv_dense(self.w.unsqueeze(0).expand(g, -1, -1), split(x), split(out), **kw)

    def __call__(self, x: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        """``out``: the activation type, or float32 rows (kept at accumulator precision)."""
        g = self._groups(x)
        if g:
            self._gemv(x, out, g)
        elif out.dtype != x.dtype:
            out.copy_(torch.mm(x, self.w.t(), out_dtype=out.dtype))
        else:
            torch.mm(x, self.w.t(), out=out)
        return out

    def activated(self, x: torch.Tensor, act: torch.Tensor, raw: torch.Tensor, kind: int, side=None) -> torch.Tensor:
        """The product with an activation behind it (`ops.dense.activate`); ``raw`` is workspace for the unfused form."""
        from ..ops import dense as ops
        g = self._groups(x)
        if g:
            self._gemv(x, act, g, act=kind, side=side)
        else:
            ops.activate(self(x, raw), act, kind, side)
        return act

    def gelu(self, x: torch.Tensor, act: torch.Tensor, gu: torch.Tensor) -> torch.Tensor:
        """act = gelu_tanh(first half) * second half of the product."""
        from ..ops import dense as ops
        return self.activated(x, act, gu, ops.ACT_GELU_MUL)
