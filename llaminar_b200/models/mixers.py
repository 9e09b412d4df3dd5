"""Mixers with sizes of their own per layer: what they keep in the cache and in the state slots, and their recurrences in plain
PyTorch (the CPU back end).

Per head, with log input gate i, log forget gate f and running maximum m (which starts at 0):

    mLSTM       m' = max(f + m, i);  S' = e^(f+m-m') S + e^(i-m') v k^T;  n' = e^(f+m-m') n + e^(i-m') k
                o = S' q / (max(|n'.q|, e^-m') + NORM_FLOOR)
    retention   S' = decay S + v k^T;  o = S' q            (lightning attention the same)

The state matrix is held as [vdim, dim]: a row per value, so that reading it out is a product with q along contiguous memory.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .config import GroupedAttention, LatentAttention, LightningAttention, MatrixLSTM, ModelConfig, ParallelMixers, Retention, WindowAttention, mixer_parts

NORM_FLOOR = 1e-6


def pad_to_multiple(n: int, of: int) -> int:
    return -(-n // of) * of


def mixer_kv_shapes(cfg: ModelConfig, head_pad=lambda dim: dim) -> list[tuple[int, ...]]:
    """Shape of every cache layer, in running order: (heads, head size), or (row width,) for latent attention."""
    out = []
    for i, _ in cfg.layer_runs():
        for p in mixer_parts(cfg.mixers[i]):
            if isinstance(p, LatentAttention):
                out.append((p.cache_width,))
            elif isinstance(p, (GroupedAttention, WindowAttention)):
                out.append((p.kv_heads, head_pad(p.head_size if isinstance(p, GroupedAttention) else p.dim)))
    return out


def conv_columns(m: GroupedAttention, head_size: int) -> int:
    """Channels of the convolution in front of an attention layer whose heads take `head_size` columns each."""
    return (m.heads + 2 * m.kv_heads) * head_size


def run_kv_layers(cfg: ModelConfig) -> list[int | None]:
    """The cache layer of every layer run (None: its mixer has no cache)."""
    out, n = [], 0
    for i, _ in cfg.layer_runs():
        cached = isinstance(cfg.mixers[i], (LatentAttention, GroupedAttention))
        out.append(n if cached else None)
        n += cached
    return out


def state_shapes_of(m, pad: int = 1, head_pad=lambda dim: dim) -> tuple[tuple[int, ...], ...]:
    if isinstance(m, GroupedAttention):             # the last projected rows: position p in place p mod taps
        return ((m.conv, conv_columns(m, head_pad(m.head_size))),)
    d, v = pad_to_multiple(m.dim, pad), pad_to_multiple(m.vdim, pad)
    if isinstance(m, MatrixLSTM):
        return (m.heads, v, d), (m.heads, d), (m.heads,)
    return ((m.heads, v, d),)


def has_state(m) -> bool:
    """Whether an elementary mixer carries something from token to token besides its cache entries."""
    return isinstance(m, (MatrixLSTM, Retention, LightningAttention)) or (isinstance(m, GroupedAttention) and m.conv > 0)


def mixer_state_shapes(cfg: ModelConfig, pad: int = 1, head_pad=lambda dim: dim) -> list[tuple[tuple[int, ...], ...]]:
    """Shapes of the state tensors of every mixer with a state, in layer order; sizes rounded up to a multiple of ``pad``."""
    return [state_shapes_of(p, pad, head_pad) for m in cfg.mixers for p in mixer_parts(m) if has_state(p)]


def mixer_columns(m) -> int:
    """Values per token between a mixer's input and output products (for the memory estimate)."""
    if isinstance(m, ParallelMixers):
        return sum(mixer_columns(p) for p in mixer_parts(m))
    if isinstance(m, WindowAttention):
        return (4 * m.heads + m.kv_heads) * m.dim
    if isinstance(m, GroupedAttention):
        return (3 * m.heads + 2 * m.kv_heads) * m.head_size + m.gate_width
    if isinstance(m, LatentAttention):
        return m.heads * (2 * m.dim + m.rot_dim + (3 if m.gated else 2) * m.vdim) + 2 * m.q_rank + 2 * m.cache_width
    if isinstance(m, (MatrixLSTM, Retention, LightningAttention)):
        return m.heads * (2 * m.dim + 4 * m.vdim)
    return 0


def soft_cap(x: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(x / cap)


def limited_pair(g: torch.Tensor, u: torch.Tensor, limit: float) -> torch.Tensor:
    """Gated pair of clamped values (see `Experts.limit`)."""
    g, u = g.clamp(max=limit), u.clamp(min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def mlstm_gates(zi: torch.Tensor, zf: torch.Tensor, cap: float) -> tuple[torch.Tensor, torch.Tensor]:
    """Log input gate and log forget gate of the gate projections (biases added)."""
    return soft_cap(zi, cap), F.logsigmoid(soft_cap(zf, cap))


def mlstm_rows(q, k, v, i, f, S, n, m):
    """New tokens of one sequence, one after the other.  q (scaled), k [T, H, d], v [T, H, e], i, f [T, H]; the state S [H, e, d],
    n [H, d], m [H] is updated in place.  Returns o [T, H, e]."""
    out = torch.empty_like(v)
    for t in range(q.shape[0]):
        top = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - top), torch.exp(i[t] - top)
        S.mul_(keep[:, None, None]).add_((add[:, None] * v[t])[:, :, None] * k[t][:, None, :])
        n.mul_(keep[:, None]).add_(add[:, None] * k[t])
        m.copy_(top)
        size = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + NORM_FLOOR
        out[t] = (S @ q[t][:, :, None])[..., 0] / size[:, None]
    return out


def retention_rows(q, k, v, decay, S):
    """As `mlstm_rows` for retention: q, k rotated, k scaled, decay [H]."""
    out = torch.empty_like(v)
    for t in range(q.shape[0]):
        S.mul_(decay[:, None, None]).add_(v[t][:, :, None] * k[t][:, None, :])
        out[t] = (S @ q[t][:, :, None])[..., 0]
    return out


def short_conv(u: torch.Tensor, before: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Causal convolution over time per channel: u [T, channels] behind the rows ``before`` [taps - 1, channels], w [taps, channels]
    with the newest tap last."""
    T, x = u.shape[0], torch.cat([before, u])
    return sum(w[j] * x[j:j + T] for j in range(w.shape[0]))
