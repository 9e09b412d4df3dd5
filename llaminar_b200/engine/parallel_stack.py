"""Decoder layers whose mixer and feed-forward run side by side on the same input, with an average over depth behind every layer.

Per layer (the residual stream h and the layers' results X are fp32, everything else bf16, or float in 32-bit mode):

    X[0] = embedding (+ position vector)                                depth_mix
    y = Wo mixer(norm1(h)) ; z = Wd a(Wu norm2(h)), or experts          engine/grouped.py, linear.py, latent.py, experts.py
    X[i + 1] = h + y + z ; h = sum of w[j] X[j] ; both norms of h       depth_mix

Both norms of the next layer come out of the update before it: they differ in their gains only.  The feed-forward runs on a stream of its
own beside the mixer (a fork and a join per layer, captured with a decode step): its weights stream from memory under the mixer's short
launches.  Between a few rows and a few hundred the sides follow one another: neither gains from sharing the machine there, and the experts'
products of more than a few rows (whose weights stream in many short pieces) lose by it.
"""
from __future__ import annotations

import torch

from .dense import DenseLinear
from .stack import AttentionStack


# batches of up to / from this many rows run both sublayers of a layer at the same time
BESIDE_FEW, BESIDE_FEW_EXPERTS, BESIDE_MANY = 64, 8, 512


class ParallelStack(AttentionStack):
    def __init__(self, model, weights):
        super().__init__(model, weights)
        c = self.cfg
        if c.loop or c.post_norms or c.embed_norm:
            raise ValueError(f"{c.arch}: parallel layers have no loops, no norms behind a sublayer and none on the embedding")
        self.positions = self.mat(weights, "position_embd.weight") if c.learned_positions else None
        self.side = torch.cuda.Stream(self.device)
        self.beside_few, self.beside_few_experts, self.beside_many = BESIDE_FEW, BESIDE_FEW_EXPERTS, BESIDE_MANY

    def build_layer(self, L, w, i: int):
        p = f"blk.{i}."
        self.build_parts(L, w, i)
        L.attn_norm = self.vec(w, p + "attn_norm.weight")
        L.ffn_norm = self.vec(w, p + "ffn_norm.weight") if L.ff or L.experts else None
        L.depth = self.vec(w, p + "depth_average.weight") if self.cfg.depth_average else None
        return L

    def alloc_workspace(self, T: int, layers) -> None:
        super().alloc_workspace(T, layers)
        c = self.cfg
        self.xn2, self.y2 = (torch.empty(T, c.d_model, dtype=self.dtype, device=self.device) for _ in range(2))
        self.past = torch.empty(c.n_layers, T, c.d_model, dtype=torch.float32, device=self.device) if c.depth_average else None

    def _norms(self, L, T: int) -> list:
        """(gain, rows) of the norms in front of a layer."""
        return [(L.attn_norm, self.xn[:T])] + ([(L.ffn_norm, self.xn2[:T])] if L.ffn_norm is not None else [])

    def run(self, fb, kv, h: torch.Tensor, layers, after_layer) -> None:
        from ..ops import dense as ops
        c, T = self.cfg, h.shape[0]
        plan = self.plan(fb, T, layers)
        past = self.past[:, :T] if self.past is not None else None
        pos = dict(z=self.positions, z_rows=fb.positions) if self.positions is not None else {}
        ops.depth_mix(h, self.embed, add=False, y_rows=fb.tokens, **pos, past=past, w=self.one if past is not None else None, norms=self._norms(layers[0], T), eps=c.rms_eps)
        for i, L in enumerate(layers):
            few = self.beside_few if L.experts is None else self.beside_few_experts
            beside = L.ffn_norm is not None and (T <= few or T >= self.beside_many)
            if beside:
                main = torch.cuda.current_stream(self.device)
                self.side.wait_stream(main)
                with torch.cuda.stream(self.side):
                    ff = self.feed_forward(L, T)
            y = L.mix.wo(self.mix(L, self.xn[:T], fb, plan, kv, i), self.y[:T])
            if beside:
                main.wait_stream(self.side)
            else:
                ff = self.feed_forward(L, T)
            ops.depth_mix(h, y, **ff, past=past, n_past=i + 1 if past is not None else 0, w=L.depth, norms=self._norms(layers[i + 1], T) if i + 1 < len(layers) else (), eps=c.rms_eps)
            after_layer(i, h)

    def feed_forward(self, L, T: int) -> dict:
        """What the residual update takes of a layer's feed-forward."""
        if L.experts is not None:
            parts, rows, weights = L.experts(self.xn2[:T])
            return dict(z=parts, z_rows=rows, z_w=weights)
        if not L.ff:
            return {}
        return dict(z=L.down(L.gate_up.activated(self.xn2[:T], self.ws("act", T, L.ff), self.ws("gu", T, L.gate_up.n_out), self.act), self.y2[:T]))

    def final_logits(self, rows: torch.Tensor, norm: torch.Tensor, head: DenseLinear, out: torch.Tensor) -> torch.Tensor:
        from ..ops import dense as ops
        xn = torch.empty(rows.shape, dtype=self.dtype, device=self.device)
        ops.depth_mix(rows, norms=[(norm, xn)], eps=self.cfg.rms_eps)
        return head(xn, out)
