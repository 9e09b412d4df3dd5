"""Mixture-of-experts feed-forward with unquantised matrices on the GPU (quantised experts: engine/moe.py).

    few rows     route (logits, choice, weights: one launch), gate|up + activation, down expert_rows: a CTA per expert and row block
    prompts      router product, choice, rows sorted by expert, gate|up + act., down     expert_grouped (tcgen05)
    32-bit mode, unusual sizes                                                           expert_plain

The chosen experts' outputs stay apart, one row per pair (token, expert); the residual norm behind the layer sums them, weighted.
"""
from __future__ import annotations

import torch

from ..models.config import Experts
from .dense import pad8, pad_to

FEW_PAIRS = 512                # pairs up to which the weights are read by `expert_rows`


class RoutedExperts:
    def __init__(self, stack, w, p: str, e: Experts):
        mat = lambda name: stack.mat(w, p + name)
        self.stack, self.e, self.ff = stack, e, pad8(e.ff)
        gate, up, down = mat("ffn_gate_exps.weight"), mat("ffn_up_exps.weight"), mat("ffn_down_exps.weight")
        self.d = d = down.shape[1]
        self.router, self.bias = mat("ffn_gate_inp.weight").contiguous(), stack.vec(w, p + "ffn_gate_inp.bias") if e.bias else None
        self.gate_up = torch.cat([pad_to(gate, e.n, self.ff, d), pad_to(up, e.n, self.ff, d)], dim=1).contiguous()        # [n, 2 ff, d]
        self.down = pad_to(down, e.n, d, self.ff).contiguous()                                                             # [n, d, ff]
        self.fast = not stack.f32 and d % 8 == 0

    def nbytes(self) -> int:
        return sum(x.numel() * x.element_size() for x in (self.router, self.gate_up, self.down))

    def __call__(self, xn: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor | None, torch.Tensor]:
        """(outputs of the pairs, row of every pair in them (None: in order), weights [tokens, top])"""
        from ..ops import experts as ops
        st, e, T = self.stack, self.e, xn.shape[0]
        P, new = T * e.top, lambda *s, dtype=xn.dtype: torch.empty(*s, dtype=dtype, device=xn.device)
        ids, weights = new(T, e.top, dtype=torch.int32), new(T, e.top, dtype=torch.float32)
        act, y = new(P, self.ff), new(P, self.d)
        if self.fast and P > FEW_PAIRS:
            logits, place, ranks = torch.mm(xn, self.router.t(), out_dtype=torch.float32), new(P, dtype=torch.int32), new(P, dtype=torch.int32)
            counts, xs = torch.zeros(e.n, dtype=torch.int32, device=xn.device), new(P, self.d)
            ops.expert_route(self.bias, ids, weights, logits=logits, counts=counts, ranks=ranks, groups=e.groups, keep=e.keep)
            ops.expert_place(xn, ids, ranks, counts, place, xs)
            ops.expert_grouped(self.gate_up, xs, counts, act, True, st.status, e.limit)
            ops.expert_grouped(self.down, act, counts, y, False, st.status)
            st.record_routing(self, ids)
            return y, place, weights
        ops.expert_route(self.bias, ids, weights, x=xn, router=self.router, groups=e.groups, keep=e.keep)
        run = ops.expert_rows if self.fast else ops.expert_plain
        run(self.gate_up, xn, ids, act, e.top, True, e.limit)
        run(self.down, act, ids, y, 1, False)
        st.record_routing(self, ids)
        return y, None, weights
