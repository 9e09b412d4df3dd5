"""Python surface of the latent-attention extension (csrc/latent_attention.cu, csrc/latent_tc.cu) and of the dense one it builds on.

As in :mod:`llaminar_b200.ops`, every call launches hand-written CUDA on the current stream; there is no fallback.  The
extension is separate from the quantised-weight kernels, so a process that serves a latent model loads only this one.
"""
from __future__ import annotations

import torch

from . import _count
from . import build as _build
from .dense import ACT_GATE, ACT_NONE, GEMV_MAX_ROWS, activate, gelu_mul, gemv_dense, gemv_fits, resid_norm, rope_angles  # noqa: F401
from .dense import bounds_status as _dense_bounds_status

_ready = False


def ext():
    global _ready
    mod = _build.load(_build.LATENT)
    if not _ready:
        from ..utils.env import debug_env
        mod.set_pdl(bool(debug_env().pdl))
        _ready = True
    return mod


def latent_prep(down, q_norm, kv_norm, angles, positions, seq_ids, block_table, cq, kv, rot_dim: int, rot_off: int, eps: float) -> None:
    """Rows [q latent | kv latent | rotated key part] of the down projection -> normed query latents ``cq`` and the tokens' rows
    of the latent cache ``kv`` (both norms, the rotation and the append in one launch)."""
    ext().latent_prep(down, q_norm, kv_norm, angles, positions, seq_ids, block_table, cq, kv, rot_dim, rot_off, eps)
    _count()


def rows_group(kv: torch.Tensor, latent: int, rot_dim: int, n_heads: int, tensor_core: bool = True) -> int:
    """Heads that share a CTA of the row kernel for these sizes: the tcgen05 form where it fits, 16 for the mma.sync form,
    0 for the plain kernel (32-bit cache, unusual sizes)."""
    if kv.dtype != torch.bfloat16:
        return 0
    e, width = ext(), kv.shape[2]
    tc = e.latent_rows_tc_heads(width, latent, rot_dim, n_heads) if tensor_core else 0
    return tc or (16 if e.latent_rows_has_kernel(width, latent) else 0)


def rows_splits(n_rows: int, n_heads: int, group: int, tensor_core: bool, max_keys: int, latent: int, capacity: int) -> int:
    """Key splits of the row kernel: about one CTA per SM (tcgen05) or two (mma.sync), whole key tiles per split, evenly
    shared, partial sums within ``capacity`` floats."""
    if group == 0:
        return 1
    groups = -(-n_heads // group)
    tiles = max_keys // (64 if tensor_core else 32) + 1             # a window that starts inside a tile touches one more
    want = max(1, min(tiles, (148 if tensor_core else 296) // max(1, n_rows * groups), 64))
    want = max(1, min(want, capacity // max(1, n_rows * groups * group * latent)))
    per = -(-tiles // want)
    return -(-tiles // per)


def latent_rows(q_lat, q, q_rot_off: int, angles, rows, positions, seq_ids, block_table, kv, rot_dim: int, window: int, scale: float,
                sink, out, part_o, part_ml, n_splits: int, group: int, status) -> None:
    """Attention of single rows over the latent cache, queries and results in the latent space ([heads, rows, latent]).
    ``group``: see `rows_group`; ``status``: device word of the tcgen05 form."""
    ext().latent_rows(q_lat, q, q_rot_off, angles, rows, positions, seq_ids, block_table, kv, rot_dim, window, scale, sink, out,
                      part_o, part_ml, n_splits, group, status)
    _count(2 if n_splits > 1 and group else 1)


def latent_gather(kv, seqs, max_k_len: int, block_table, out) -> None:
    """The cache rows of the keys that the sequences of ``seqs`` see, one after the other."""
    ext().latent_gather(kv, seqs, max_k_len, block_table, out)
    _count()


def latent_chunk(q, angles, k, v, lat, rot_off: int, seqs, max_q_len: int, out, dim: int, rot: int, vdim: int, window: int,
                 scale: float, sink, status=None, gate=None) -> None:
    """Attention of prompt chunks on keys and values written out per head and the shared rotated parts in ``lat``.  With
    ``status`` the tcgen05 form runs, which takes the values transposed ([heads * vdim, keys]).  ``gate`` [tokens, heads * vdim]: the result times its
    sigmoid."""
    ext().latent_chunk(q, angles, k, v, lat, rot_off, seqs, max_q_len, out, dim, rot, vdim, window, scale, sink, status, gate)
    _count()


def chunk_has_kernel(dk: int, dv: int) -> bool:
    return bool(ext().latent_chunk_has_kernel(dk, dv))


def chunk_tc_fits(dim: int, rot: int, vdim: int) -> bool:
    return bool(ext().latent_chunk_tc_fits(dim, rot, vdim))


def bounds_status(reset: bool = True) -> int:
    return int(ext().bounds_status(bool(reset))) | _dense_bounds_status(reset)
