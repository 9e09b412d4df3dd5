"""Python surface of the experts extension (csrc/experts.cu, experts_tc.cu): mixture-of-experts feed-forwards with unquantised matrices.

As in :mod:`llaminar_b200.ops`, every call launches hand-written CUDA on the current stream; there is no fallback.  A pair is (token,
one of its chosen experts): pair p belongs to token p // top.
"""
from __future__ import annotations

import torch

from . import _count
from . import build as _build

_ready = False


def ext():
    global _ready
    mod = _build.load(_build.EXPERTS)
    if not _ready:
        from ..utils.env import debug_env
        mod.set_pdl(bool(debug_env().pdl))
        _ready = True
    return mod


def max_pairs() -> int:
    """Most pairs that `expert_rows` takes."""
    return ext().MAX_PAIRS


def expert_route(bias, ids, weights, x=None, router=None, logits=None, counts=None, ranks=None, groups: int = 1, keep: int = 1) -> None:
    """Router logits (x router^T, or given) + bias in 32-bit -> the ``top`` largest (``ids`` [tokens, top]) and the softmax over just
    those.  With several ``groups`` of neighbours only the experts of the ``keep`` groups with the largest logits count.  ``counts`` (zeroed) and ``ranks``: pairs per expert, and the number of a pair among those of its expert.  One launch."""
    ext().expert_route(x, router, logits, bias, ids, weights, counts, ranks, groups, keep)
    _count()


def expert_place(x, ids, ranks, counts, place, xs) -> None:
    """xs[place[pair]] = x[token of the pair], sorted by expert."""
    ext().expert_place(x, ids, ranks, counts, place, xs)
    _count()


def expert_rows(w, x, ids, out, div: int, pair_act: bool, limit: float = 0.0) -> None:
    """out[pair] = x[pair // div] w[ids[pair]]^T for few pairs (bf16); ``pair_act``: w stacks gate and up, out = silu(gate) * up, or
    with a ``limit`` g sigmoid(1.702 g) (u + 1) of the clamped values."""
    ext().expert_rows(w, x, ids, out, div, pair_act, limit)
    _count()


def expert_plain(w, x, ids, out, div: int, pair_act: bool, limit: float = 0.0) -> None:
    """As `expert_rows` in float arithmetic: 32-bit mode, and sizes without a tensor-core kernel."""
    ext().expert_plain(w, x, ids, out, div, pair_act, limit)
    _count()


def expert_grouped(w, x, counts, out, pair_act: bool, status, limit: float = 0.0) -> None:
    """The same product for rows sorted by expert (tcgen05): ``counts`` rows of each."""
    ext().expert_grouped(w, x, counts, out, pair_act, status, limit)
    _count()


def grouped_fits(n: int, k: int, experts: int) -> bool:
    return bool(ext().expert_grouped_fits(n, k, experts))


def bounds_status(reset: bool = True) -> int:
    return int(ext().bounds_status(bool(reset)))
