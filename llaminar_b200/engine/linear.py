"""Lightning attention on the GPU: a layer's weights and its kernel sequence between the input norm and the output product.

    [q | k | v | gate] = W xn                                   one product (decode steps keep it in float)
    state, outputs of the heads                                 linear_rows (silu as it reads), or silu in place and linear_chunk (prompts)
    norm over all heads, output gate                            joint_gate

Head sizes are zero-padded to multiples of 8 when the weights are loaded.
"""
from __future__ import annotations

import torch

from ..models.config import LightningAttention
from .dense import DenseLinear, pad8, pad_to

SHORT_ROWS = 4                 # batches of portions up to this long advance the recurrence row by row


class LightningMixer:
    """One layer's lightning attention.  ``stack``: the `AttentionStack` it belongs to; ``state``: its place among the layers with one."""

    def __init__(self, stack, w, p: str, m: LightningAttention, state: int):
        self.stack, self.m, self.state, H = stack, m, state, m.heads
        self.dim, self.vdim = d, v = pad8(m.dim), pad8(m.vdim)

        def heads(name: str, size: int) -> torch.Tensor:
            x = stack.mat(w, p + name).view(H, -1, stack.cfg.d_model)
            return pad_to(x, H, size, x.shape[2]).view(H * size, -1)

        self.proj = DenseLinear(torch.cat([heads("lin_q.weight", d), heads("lin_k.weight", d), heads("lin_v.weight", v), heads("lin_g.weight", v)]))
        self.offs = [0, H * d, 2 * H * d, 2 * H * d + H * v]
        self.norm = pad_to(stack.vec(w, p + "lin_norm.weight").view(H, -1), H, v).reshape(-1).contiguous()
        self.decay = torch.tensor(m.decay, dtype=torch.float32, device=stack.device)
        o = stack.mat(w, p + "lin_output.weight").view(-1, H, m.vdim)
        self.wo = DenseLinear(pad_to(o, o.shape[0], H, v).view(o.shape[0], -1))

    def nbytes(self) -> int:
        return self.proj.nbytes() + self.wo.nbytes()

    def workspace(self) -> dict[str, int]:
        return {"rows": self.proj.n_out, "raw": self.wo.k, "o": self.wo.k}

    def __call__(self, xn: torch.Tensor, fb, plan, kv, kv_layer=None) -> torch.Tensor:
        """Normed input rows -> the gated heads, input of the output product."""
        from ..ops import dense as dense_ops
        from ..ops import mixers as ops
        st, m, T, eps = self.stack, self.m, xn.shape[0], self.stack.cfg.rms_eps
        rows = self.proj(xn, st.ws("rows", T, self.proj.n_out, torch.float32 if fb.is_decode else None))
        raw, out = st.ws("raw", T, self.wo.k, rows.dtype), st.ws("o", T, self.wo.k)
        args = (rows, self.offs, None, self.decay, None, 1.0, 1.0, None if fb.is_decode else fb.cu_q, fb.positions, fb.state_slots,
                kv.hybrid.layers[self.state], m.vdim, None, False)
        if plan.chunks is not None and ops.linear_chunk_fits(self.dim, self.vdim):
            qkv = rows[:, :self.offs[3]]
            dense_ops.activate(qkv, qkv, dense_ops.ACT_SILU)
            ops.linear_chunk(*args, out, eps, plan.chunks, raw, st.status, only_raw=True)
        else:
            ops.linear_rows(*args, raw, eps, silu_in=True, raw=True)
        ops.joint_gate(raw, rows, self.offs[3], self.norm, m.heads * m.vdim, out, eps)
        return out
