"""Python surface of the mixers extension (csrc/mixers.cu, linear_tc.cu): linear attention with a recurrent state.

As in :mod:`llaminar_b200.ops`, every call launches hand-written CUDA on the current stream; there is no fallback.
"""
from __future__ import annotations

import torch

from . import _count
from . import build as _build

_ready = False


def ext():
    global _ready
    mod = _build.load(_build.MIXERS)
    if not _ready:
        from ..utils.env import debug_env
        mod.set_pdl(bool(debug_env().pdl))
        _ready = True
    return mod


def linear_rows(rows, offs, gates, decay, angles, q_scale: float, k_scale: float, cu, positions, slots, state, true_vdim: int, norm_w,
                silu: bool, out, eps: float, silu_in: bool = False, raw: bool = False) -> None:
    """mLSTM (``gates``: float rows of gate projections, input biases, forget biases, cap) or a fixed ``decay`` (retention, lightning
    attention), the rows of a sequence one after the other; ``cu`` None: one row per sequence.  The state of ``slots`` is advanced in
    place.  ``silu_in``: q, k and v pass through silu first; ``raw``: the outputs without norm and gate."""
    g = gates or (None, None, None, 1.0)
    ext().linear_rows(rows, list(offs), *g, decay, angles, q_scale, k_scale, cu, positions, slots, list(state), true_vdim, norm_w, silu, out, eps, silu_in, raw)
    _count()


def chunk_tables(cu: list[int], device) -> tuple[torch.Tensor, torch.Tensor]:
    """How the chunk kernels cut a packed batch whose sequence b has rows cu[b] .. cu[b + 1]: (first row, rows, sequence, last of it)
    per chunk and (first chunk, chunks, 0, 0) per sequence."""
    size = ext().LINEAR_CHUNK
    chunks, seqs = [], []
    for b in range(len(cu) - 1):
        first = len(chunks)
        for r in range(cu[b], cu[b + 1], size):
            n = min(size, cu[b + 1] - r)
            chunks.append((r, n, b, int(r + n == cu[b + 1])))
        seqs.append((first, len(chunks) - first, 0, 0))
    it = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
    return it(chunks), it(seqs)


def linear_chunk_fits(dim: int, vdim: int) -> bool:
    return bool(ext().linear_chunk_fits(dim, vdim))


def linear_chunk(rows, offs, gates, decay, angles, q_scale: float, k_scale: float, cu, positions, slots, state, true_vdim: int, norm_w,
                 silu: bool, out, eps: float, tables, raw, status, only_raw: bool = False) -> None:
    """As `linear_rows` for prompts in bf16, chunk-parallel on the tensor cores.  ``tables``: see `chunk_tables`; ``raw``: workspace
    like ``out``, with ``only_raw`` the result (without norm and gate; ``out`` is not written)."""
    g = gates or (None, None, None, 1.0)
    chunks, seqs = tables
    _, h, v, d = state[0].shape
    n = chunks.shape[0]
    f = lambda *s: torch.empty(*s, dtype=torch.float32, device=rows.device)
    ext().linear_chunk(rows, list(offs), *g, decay, angles, q_scale, k_scale, cu, positions, slots, list(state), true_vdim, norm_w, silu, out, eps,
                       chunks, seqs, f(n, h, v, d), f(n, h, d), f(n, h, 4), f(n, h, ext().LINEAR_CHUNK, 4) if gates else None, raw, status, only_raw)
    _count(4 if v > 256 and not only_raw else 3)


def joint_gate(o, rows, g_off: int, norm_w, true_n: int, out, eps: float) -> None:
    """out = o / rms(o) * norm_w * sigmoid(gate columns of ``rows``), the root mean square over a whole row (``true_n`` values that are
    not padding)."""
    ext().joint_gate(o, rows, g_off, norm_w, true_n, out, eps)
    _count()


def bounds_status(reset: bool = True) -> int:
    return int(ext().bounds_status(bool(reset)))
