"""Python surface of the mixers extension (csrc/mixers.cu, linear_tc.cu, attention.cu, attention_tc.cu): grouped-query attention with a
sliding window, sinks and an output gate, and linear attention with a recurrent state.

As in :mod:`llaminar_b200.ops`, every call launches hand-written CUDA on the current stream; there is no fallback.
"""
from __future__ import annotations

import torch

from . import _attn_tc_default, _count
from . import build as _build

DECODE_GROUP = 16              # query heads per key head that the decode kernel takes
HEAD_SIZES = (64, 128)         # of the tensor-core attention kernels
_ready = False


def ext():
    global _ready
    mod = _build.load(_build.MIXERS)
    if not _ready:
        from ..utils.env import debug_env
        mod.set_pdl(bool(debug_env().pdl))
        _ready = True
    return mod


def attn_prep(rows, q_off: int, k_off: int, v_off: int, q_norm, k_norm, positions, seq_ids, block_table, q_out, kv, true_dim: int, eps: float) -> None:
    """Projected rows -> normed queries [tokens, heads, dim] and the tokens' entries of the paged cache (both norms over all heads
    of a projection, and the append, in one launch).  ``v_off`` = ``k_off``: the values are the keys before their norm."""
    ext().attn_prep(rows, q_off, k_off, v_off, q_norm, k_norm, positions, seq_ids, block_table, q_out, kv, true_dim, eps)
    _count()


def window_plain(q, kv, out, positions, seq_ids, block_table, window: int, scale: float, sink, gate) -> None:
    """Attention of any rows in float arithmetic: 32-bit mode, and shapes without a tensor-core kernel."""
    ext().window_plain(q, kv, out, positions, seq_ids, block_table, window, scale, sink, gate)
    _count()


def decode_splits(batch: int, kv_heads: int, dim: int, max_pages: int, window: int, scratch) -> int:
    """Key splits of the decode kernel: about two CTAs per SM, at least two pages each, partial sums within the scratch."""
    pages = min(max_pages, window // 64 + 2) if window else max_pages
    n = max(1, min(16, 296 // max(1, batch * kv_heads), pages // 2))
    n = min(n, scratch.part_o.numel() // (batch * kv_heads * 16 * dim), scratch.part_ml.numel() // (batch * kv_heads * 32))
    return max(1, n) if batch * kv_heads <= scratch.attn_tickets.numel() else 1


def attn_decode(q, kv, out, block_table, seq_lens, scale: float, n_splits: int, window: int, sink, gate, scratch) -> None:
    """One row per sequence.  ``gate``: float rows whose sigmoid multiplies the result."""
    ext().attn_decode(q, kv, out, block_table, seq_lens, scratch.part_o, scratch.part_ml, scratch.attn_tickets, scale, n_splits, window, sink, gate)
    _count()


def attn_prefill(q, kv, out, block_table, cu_q, ctx_lens, scale: float, max_q_len: int, window: int, sink, gate, status=None) -> None:
    """Portions of prompts; with ``status`` the tcgen05 form."""
    ext().attn_prefill(q, kv, out, block_table, cu_q, ctx_lens, scale, max_q_len, window, sink, gate, status)
    _count()


def prefill_tc(dim: int, max_q_len: int) -> bool:
    return dim == 128 and max_q_len >= 128 and _attn_tc_default()


def linear_rows(rows, offs, gates, decay, angles, q_scale: float, k_scale: float, cu, positions, slots, state, true_vdim: int, norm_w,
                silu: bool, out, eps: float) -> None:
    """mLSTM (``gates``: float rows of gate projections, input biases, forget biases, cap) or retention (``decay``), the rows of a
    sequence one after the other; ``cu`` None: one row per sequence.  The state of ``slots`` is advanced in place."""
    g = gates or (None, None, None, 1.0)
    ext().linear_rows(rows, list(offs), *g, decay, angles, q_scale, k_scale, cu, positions, slots, list(state), true_vdim, norm_w, silu, out, eps)
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
                 silu: bool, out, eps: float, tables, raw, status) -> None:
    """As `linear_rows` for prompts in bf16, chunk-parallel on the tensor cores.  ``tables``: see `chunk_tables`; ``raw``: workspace
    like ``out``."""
    g = gates or (None, None, None, 1.0)
    chunks, seqs = tables
    _, h, v, d = state[0].shape
    n = chunks.shape[0]
    f = lambda *s: torch.empty(*s, dtype=torch.float32, device=rows.device)
    ext().linear_chunk(rows, list(offs), *g, decay, angles, q_scale, k_scale, cu, positions, slots, list(state), true_vdim, norm_w, silu, out, eps,
                       chunks, seqs, f(n, h, v, d), f(n, h, d), f(n, h, 4), f(n, h, ext().LINEAR_CHUNK, 4) if gates else None, raw, status)
    _count(4 if v > 256 else 3)


def bounds_status(reset: bool = True) -> int:
    return int(ext().bounds_status(bool(reset)))
