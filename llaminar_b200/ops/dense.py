"""Python surface of the dense extension (csrc/dense_ops.cu): what models with unquantised matrices share.

As in :mod:`llaminar_b200.ops`, every call launches hand-written CUDA on the current stream; there is no fallback.  The
extension is separate from the quantised-weight kernels, so a process that serves such a model does not load those.
"""
from __future__ import annotations

import torch

from . import _count
from . import build as _build

GEMV_MAX_ROWS = 8
ACT_NONE, ACT_GELU_MUL, ACT_RELU2, ACT_GELU_SIDE, ACT_SILU_MUL, ACT_GATE, ACT_GELU, ACT_SILU = range(8)
_ready = False


def ext():
    global _ready
    mod = _build.load(_build.DENSE)
    if not _ready:
        from ..utils.env import debug_env
        mod.set_pdl(bool(debug_env().pdl))
        _ready = True
    return mod


def resid_norm(h, y=None, w_post=None, *, add=True, y_rows=None, w_next=None, xn=None, copy0=None, copy1=None, eps: float, y2=None,
               w_y=None, w_y2=None, factor: float = 1.0, center_post: bool = False, center_next: bool = False, y_w=None) -> None:
    """h = (h if add) + norm(y) * w_post (``y`` None: h is only read; ``y_rows`` gathers rows of y; ``w_post`` None: y * factor),
    then xn = norm(h) * w_next and copies of h in the activation type.  With ``y2``, y stands for half the sum of RMSNorm(y) * w_y
    and RMSNorm(y2) * w_y2; with ``y_w`` [tokens, parts] for the sum of a token's rows of y (all of them, or those ``y_rows`` names) times their
    weights.  The norms are RMSNorms, or with ``center_post`` / ``center_next`` layer norms without a bias.  One launch."""
    ext().resid_norm(y, y_rows, w_post, h, add, w_next, xn, copy0, copy1, eps, y2, w_y, w_y2, factor, center_post, center_next, y_w)
    _count()


def depth_mix(h, y=None, z=None, *, add=True, y_rows=None, z_rows=None, z_w=None, past=None, n_past: int = 0, w=None, norms=(), eps: float) -> None:
    """x = (h if add) + y + z, rows of either gathered by ``y_rows`` / ``z_rows``, z the sum of a token's rows times ``z_w`` [tokens,
    parts] if given; h = sum of w[j] past[j] over j < n_past plus w[n_past] x, and past[n_past] = x if ``past`` [streams, tokens, d] has that
    stream.  ``norms``: up to two (gain, output) pairs of RMSNorms of h, gains of one value or of d.  One launch."""
    (g0, x0), (g1, x1) = (*norms, (None, None), (None, None))[:2]
    ext().depth_mix(h, add, y, y_rows, z, z_rows, z_w, past, n_past, w, g0, x0, g1, x1, eps)
    _count()


def activate(x: torch.Tensor, act: torch.Tensor, kind: int, side=None) -> None:
    """act = gelu_tanh(x[:, :n]) * x[:, n:] (ACT_GELU_MUL), the same with silu (ACT_SILU_MUL), both without a second half (ACT_GELU, ACT_SILU),
    squared relu (ACT_RELU2), gelu_tanh(x) times
    columns of each token's row of a table (ACT_GELU_SIDE; ``side``: table, first column, columns, tokens), or x times the sigmoid of
    those columns of the row itself (ACT_GATE; tokens None).  ``act`` may be ``x``, except for the pairs."""
    ext().activate(x, act, kind, *(side or (None, 0, 0, None)))
    _count()


def gelu_mul(gu: torch.Tensor, act: torch.Tensor) -> None:
    """act = gelu_tanh(gu[:, :ff]) * gu[:, ff:]"""
    activate(gu, act, ACT_GELU_MUL)


def rope_angles(positions: torch.Tensor, freqs: torch.Tensor, magnitude: float, out: torch.Tensor) -> None:
    """out[t, i] = magnitude * (cos, sin)(positions[t] * freqs[i]); freqs in double precision."""
    ext().rope_angles(positions, freqs, magnitude, out)
    _count()


def gemv_fits(w: torch.Tensor, x: torch.Tensor) -> bool:
    """Whether `gemv_dense` takes this product: few bf16 rows, 16-byte rows."""
    k = w.shape[-1]
    return (w.dtype == torch.bfloat16 and x.shape[-2] <= GEMV_MAX_ROWS and k % 8 == 0 and x.stride(-2) % 8 == 0 and w.stride(-2) % 8 == 0
            and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)


def gemv_dense(w, x, out, gelu: bool = False, act: int = ACT_NONE, side=None) -> None:
    """out[z] = x[z] @ w[z]^T for at most eight bf16 rows; ``act`` (see `activate`): applied to the result (a gate's columns run over
    all z); ``gelu``: w stacks gate and up, out = gelu_tanh(gate) * up."""
    ext().gemv_dense(w, x, out, ACT_GELU_MUL if gelu else act, *(side or (None, 0, 0, None)))
    _count()


def bounds_status(reset: bool = True) -> int:
    return int(ext().bounds_status(bool(reset)))
