"""Python surface of the grouped-attention extension (csrc/grouped.cu, attention.cu, attention_tc.cu): grouped-query attention with
windows, chunks, sinks, soft caps and output gates.

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
    mod = _build.load(_build.GROUPED)
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


def head_prep(rows, q_off: int, k_off: int, v_off: int, q_norm, k_norm, angles, positions, seq_ids, block_table, q_out, kv, true_dim: int, eps: float) -> None:
    """Projected rows -> queries [tokens, heads, dim] and the tokens' entries of the paged cache: queries and keys normed per head and
    rotated (pairs (i, i + half)), values as they are.  One launch."""
    ext().head_prep(rows, q_off, k_off, v_off, q_norm, k_norm, angles, positions, seq_ids, block_table, q_out, kv, true_dim, eps)
    _count()


def conv_prep(rows, taps, ring, slots, cu, angles, q_gain, first, share, positions, seq_ids, block_table, q_out, kv) -> None:
    """Projected rows [q | k | v | ...] -> queries [tokens, heads, dim] and the tokens' entries of the paged cache, every channel passed
    through a causal convolution over time (``taps`` [n, channels], the last rows of each sequence in its slot of ``ring``), queries and
    keys rotated, queries times ``q_gain`` of their head.  ``first`` [tokens, kv heads, values]: receives the values, or with ``share``
    brings those of an earlier layer that are mixed in.  One launch; with ``cu`` (portions of prompts) another one for the ring."""
    ext().conv_prep(rows, taps, ring, slots, cu, angles, q_gain, first, share, positions, seq_ids, block_table, q_out, kv)
    _count(1 if cu is None or taps.shape[0] == 1 else 2)


def attn_plain(q, kv, out, positions, seq_ids, block_table, window: int, scale: float, sink, gate, chunk: int = 0, softcap: float = 0.0) -> None:
    """Attention of any rows in float arithmetic: 32-bit mode, and shapes without a tensor-core kernel."""
    ext().attn_plain(q, kv, out, positions, seq_ids, block_table, window, scale, sink, gate, chunk, softcap)
    _count()


def decode_splits(batch: int, kv_heads: int, dim: int, max_pages: int, window: int, scratch, chunk: int = 0) -> int:
    """Key splits of the decode kernel: about two CTAs per SM, at least two pages each, partial sums within the scratch."""
    pages = min([max_pages] + [n // 64 + 2 for n in (window, chunk) if n])
    n = max(1, min(16, 296 // max(1, batch * kv_heads), pages // 2))
    n = min(n, scratch.part_o.numel() // (batch * kv_heads * 16 * dim), scratch.part_ml.numel() // (batch * kv_heads * 32))
    return max(1, n) if batch * kv_heads <= scratch.attn_tickets.numel() else 1


def attn_decode(q, kv, out, block_table, seq_lens, scale: float, n_splits: int, window: int, sink, gate, scratch, chunk: int = 0,
                softcap: float = 0.0) -> None:
    """One row per sequence.  ``gate``: float rows whose sigmoid multiplies the result, [rows, heads * dim] or [rows, heads]."""
    ext().attn_decode(q, kv, out, block_table, seq_lens, scratch.part_o, scratch.part_ml, scratch.attn_tickets, scale, n_splits, window, sink, gate,
                      chunk, softcap)
    _count()


def attn_prefill(q, kv, out, block_table, cu_q, ctx_lens, scale: float, max_q_len: int, window: int, sink, gate, status=None, chunk: int = 0,
                 softcap: float = 0.0) -> None:
    """Portions of prompts; with ``status`` the tcgen05 form."""
    ext().attn_prefill(q, kv, out, block_table, cu_q, ctx_lens, scale, max_q_len, window, sink, gate, status, chunk, softcap)
    _count()


def prefill_tc(dim: int, max_q_len: int) -> bool:
    return dim == 128 and max_q_len >= 128 and _attn_tc_default()


def bounds_status(reset: bool = True) -> int:
    return int(ext().bounds_status(bool(reset)))
