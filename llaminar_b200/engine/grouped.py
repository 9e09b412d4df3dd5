"""Grouped-query attention with norms per head or short convolutions, rotation, windows or chunks, soft caps and output gates on the GPU: a
layer's weights and its kernel sequence between the input norm and the output product.

    [q | k | v | gate] = W xn                                   one product (decode steps keep it in float)
    norms, rotation, cache append                               head_prep, or
    convolution, rotation, mixed values, cache append           conv_prep
    attention, output gate                                      attn_decode, attn_prefill, or attn_plain (32-bit mode, unusual sizes)

Heads are zero-padded to the kernels' sizes when the weights are loaded.  Rotated parts are stored in the order in which pair i is
(i, i + half): queries, keys and their gains alike, so the scores are the same.
"""
from __future__ import annotations

import torch

from ..models.config import GroupedAttention
from .dense import DenseLinear, pad8, pad_to


def padded_head(size: int, f32: bool) -> int:
    """Head size of the attention kernels for heads of ``size`` values."""
    from ..ops import grouped as ops
    if f32 or size > max(ops.HEAD_SIZES):
        return pad8(size)
    return min(s for s in ops.HEAD_SIZES if s >= size)


class GroupedMixer:
    """One layer's grouped-query attention.  ``stack``: the `AttentionStack` it belongs to."""

    def __init__(self, stack, w, p: str, m: GroupedAttention, state: int = 0):
        """``state``: place among the layers with a state (the convolution's last rows)."""
        D = self.dim = padded_head(m.head_size, stack.f32)
        if bool(m.conv) == m.qk_norm or (m.conv == 0 and (m.temperature or m.value_mix)):
            raise ValueError("grouped attention: either norms per head, or convolutions (with temperatures and mixed values)")
        self.stack, self.m, self.state = stack, m, state
        order = torch.tensor(m.rotary.halves_order(m.dim), device=stack.device)

        def heads(name: str, n: int, size: int, order=None) -> torch.Tensor:
            x = stack.mat(w, p + name).view(n, size, -1)
            x = x if order is None else x[:, order]
            return pad_to(x, n, D, x.shape[2]).view(n * D, -1)

        gain = lambda name: pad_to(stack.vec(w, p + name)[order], D)
        rows = [heads("attn_q.weight", m.heads, m.dim, order), heads("attn_k.weight", m.kv_heads, m.dim, order), heads("attn_v.weight", m.kv_heads, m.vdim)]
        if m.gate == "head":
            g = stack.mat(w, p + "attn_gate.weight")
            rows.append(pad_to(g, pad8(m.heads), g.shape[1]))
        elif m.gate:
            rows.append(heads("attn_gate.weight", m.heads, m.vdim))
        self.offs = [0, m.heads * D, (m.heads + m.kv_heads) * D, (m.heads + 2 * m.kv_heads) * D]
        self.gate_cols = {"": 0, "head": m.heads, "value": m.heads * D}[m.gate]
        self.proj = DenseLinear(torch.cat(rows))
        if m.qk_norm:
            self.q_norm, self.k_norm = gain("attn_q_norm.weight"), gain("attn_k_norm.weight")
        if m.conv:
            def taps(name: str, n: int, size: int, order=None) -> torch.Tensor:
                x = w[p + name].to_float().to(stack.device).view(n, size, -1)
                x = x if order is None else x[:, order]
                return pad_to(x, n, D, x.shape[2]).view(n * D, -1)
            self.taps = torch.cat([taps("attn_q_conv.weight", m.heads, m.dim, order), taps("attn_k_conv.weight", m.kv_heads, m.dim, order),
                                   taps("attn_v_conv.weight", m.kv_heads, m.vdim)]).t().contiguous()
        self.q_gain = stack.vec(w, p + "attn_temperature.weight") if m.temperature else None
        self.share = stack.vec(w, p + "attn_value_mix.weight") if m.value_mix else None
        o = stack.mat(w, p + "attn_output.weight").view(-1, m.heads, m.vdim)
        self.wo = DenseLinear(pad_to(o, o.shape[0], m.heads, D).view(o.shape[0], -1))
        self.sink = torch.zeros(m.heads, device=stack.device) if m.null_key else None       # the key with score 0 is a sink of logit 0
        self.rot = stack.rotation(m.rotary)

    def nbytes(self) -> int:
        return self.proj.nbytes() + self.wo.nbytes()

    def workspace(self) -> dict[str, int]:
        return {"rows": self.proj.n_out, "q": self.m.heads * self.dim, "o": self.wo.k, **({"values": 2 * self.m.kv_heads * pad8(self.m.vdim)} if self.m.value_mix else {})}

    def _prep(self, rows, fb, plan, kv, kv_layer, q) -> None:
        """Queries, and the cache entries of the tokens, from the projected rows."""
        from ..ops import grouped as ops
        st, m = self.stack, self.m
        if not m.conv:
            ops.head_prep(rows, *self.offs[:3], self.q_norm, self.k_norm, plan.angles[self.rot], fb.positions, fb.seq_ids, fb.block_table, q, kv_layer, m.dim, st.cfg.rms_eps)
            return
        values, share = plan.values, self.share
        if m.value_mix and values is None:                              # the first such layer: its values are kept for the others
            size = pad8(m.vdim)
            values, share = st.ws("values", rows.shape[0], m.kv_heads * size, torch.float32).view(-1, m.kv_heads, size), None
            plan.values = values
        ops.conv_prep(rows, self.taps, kv.hybrid.layers[self.state][0], fb.state_slots, None if fb.is_decode else fb.cu_q, plan.angles[self.rot], self.q_gain,
                      values if m.value_mix else None, share, fb.positions, fb.seq_ids, fb.block_table, q, kv_layer)

    def __call__(self, xn: torch.Tensor, fb, plan, kv, kv_layer: torch.Tensor) -> torch.Tensor:
        """Normed input rows -> the gated heads, input of the output product."""
        from ..ops import grouped as ops
        st, m, T, D = self.stack, self.m, xn.shape[0], self.dim
        H, G = m.heads, m.kv_heads
        rows = self.proj(xn, st.ws("rows", T, self.proj.n_out, torch.float32 if fb.is_decode else None))
        q, o = st.ws("q", T, H * D).view(T, H, D), st.ws("o", T, H * D)
        self._prep(rows, fb, plan, kv, kv_layer, q)
        gate = rows[:, self.offs[3]:self.offs[3] + self.gate_cols] if m.gate else None
        mask = dict(chunk=m.chunk, softcap=m.softcap)
        fits = not st.f32 and D in ops.HEAD_SIZES
        if fits and fb.is_decode and H // G <= ops.DECODE_GROUP:
            splits = ops.decode_splits(T, G, D, fb.block_table.shape[1], m.window, st.scratch, m.chunk)
            ops.attn_decode(q, kv_layer, o, fb.block_table, fb.seq_lens, m.scale, splits, m.window, self.sink, gate, st.scratch, **mask)
        elif fits and not fb.is_decode:
            tc = st.prefill_tc and ops.prefill_tc(D, fb.max_q_len)
            ops.attn_prefill(q, kv_layer, o, fb.block_table, fb.cu_q, fb.ctx_lens, m.scale, fb.max_q_len, m.window, self.sink, gate, st.status if tc else None, **mask)
        else:
            ops.attn_plain(q, kv_layer, o, fb.positions, fb.seq_ids, fb.block_table, m.window, m.scale, self.sink, gate, **mask)
        return o
