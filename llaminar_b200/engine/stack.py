"""Decoder layers of latent, grouped or lightning attention with a dense or routed feed-forward each: weights, workspace and the kernel sequence of
`CudaModel` for such models.

Per layer (the residual stream h is fp32, everything else bf16, or float in 32-bit mode):

    o = attention(xn)                                           engine/latent.py, grouped.py, linear.py
    y = Wo o ; h += norm(y) ; xn = norm(h)                      resid_norm
    act = a(Wg xn) * (Wu xn) ; y = Wd act                       fused into the product up to eight rows; or engine/experts.py
    h += norm(y) ; xn = norm(h) of the next layer               resid_norm (sums the chosen experts' rows first)

Layers of a loop run several times, each pass behind a projection of [h | embedding].  Matrix products run on `gemv_dense` up to eight
rows and on cuBLAS above.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..models.config import GroupedAttention, LatentAttention, LightningAttention, Rotary
from ..models.mixers import has_state, mixer_kv_shapes, mixer_state_shapes, run_kv_layers
from .dense import DenseLinear
from .experts import RoutedExperts
from .grouped import GroupedMixer, padded_head
from .latent import PART_FLOATS, LatentMixer, LatentPlan
from .linear import SHORT_ROWS, LightningMixer


@dataclass
class StackPlan:
    """What the layers of one forward call share."""
    angles: list[torch.Tensor]                       # per distinct rotation: [T, dims/2, 2]
    latent: LatentPlan | None = None
    chunks: tuple | None = None                      # how the chunk kernels of a recurrence cut the batch (None: row after row)
    values: torch.Tensor | None = None               # of the first layer whose values later ones mix in


class AttentionStack:
    def __init__(self, model, weights):
        from ..ops import dense as ops
        c = self.cfg = model.cfg
        self.device, self.dtype, self.model = model.device, model.dtype, model
        self.f32 = self.dtype == torch.float32
        self.rows_tc = self.chunk_tc = self.prefill_tc = True           # tcgen05 forms of the attention kernels where the sizes fit
        # sums stay in 32 bits: no TF32 operands in 32-bit mode, no 16-bit reduction of split products otherwise
        if self.f32:
            torch.backends.cuda.matmul.allow_tf32 = False
        else:
            torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        self.embed = self.mat(weights, "token_embd.weight")
        self.embed_norm = self.vec(weights, "token_embd_norm.weight") if c.embed_norm else None
        self.loop_in = DenseLinear(self.mat(weights, "loop_in.weight")) if c.loop else None
        self.loop_step = self.mat(weights, "loop_step.weight") if c.loop_steps else None
        self.act = {"silu": ops.ACT_SILU_MUL, "gelu_tanh": ops.ACT_GELU_MUL, "gelu_up": ops.ACT_GELU}[c.ffn_act]
        from .. import ops as base
        self.scratch = base.scratch_for(self.device)
        self.status = self.scratch.status                               # word that a kernel sets when a bounded wait runs out
        self.runs = c.layer_runs()                                      # looped layers have a cache layer per pass
        head_pad = lambda size: padded_head(size, self.f32)
        self.kv_layer_shapes, self.kv_index = mixer_kv_shapes(c, head_pad), run_kv_layers(c)
        self.state_shapes = mixer_state_shapes(c, 8, head_pad)
        self.state_index = [sum(has_state(m) for m in c.mixers[:i]) for i in range(c.n_layers)]
        self.n_kv_layers = len(self.kv_layer_shapes)
        self.linear_tc = True                                           # tcgen05 form of the recurrence over prompts where the sizes fit
        self.rotaries: list[Rotary] = []
        self.freqs: list[torch.Tensor] = []
        self.has_latent, self.has_linear = (any(isinstance(m, kind) for m in c.mixers) for kind in (LatentAttention, LightningAttention))
        self.one = torch.ones(1, dtype=torch.float32, device=self.device)

    def mat(self, w, name: str) -> torch.Tensor:
        return w[name].to_float().to(self.device).to(self.dtype)

    def vec(self, w, name: str) -> torch.Tensor:
        return w[name].to_float().to(device=self.device, dtype=torch.float32).contiguous()

    def rotation(self, r: Rotary) -> int:
        """Index of a rotation's angles in a plan."""
        if r not in self.rotaries:
            self.rotaries.append(r)
            self.freqs.append(torch.tensor(r.frequencies(), dtype=torch.float64, device=self.device))
        return self.rotaries.index(r)

    def head_matrix(self, w) -> torch.Tensor:
        return self.embed if self.cfg.tie_embeddings else self.mat(w, "output.weight")

    # -- weights ---------------------------------------------------------------------------------------------
    def build_parts(self, L, w, i: int) -> None:
        """A layer's mixer and feed-forward."""
        c, m, p = self.cfg, self.cfg.mixers[i], f"blk.{i}."
        L.index = i
        if isinstance(m, LightningAttention):
            L.mix = LightningMixer(self, w, p, m, self.state_index[i])
        else:
            L.mix = GroupedMixer(self, w, p, m, self.state_index[i]) if isinstance(m, GroupedAttention) else LatentMixer(self, w, p, m)
        L.ff, e = c.ff_width(i), c.experts_of(i)
        L.experts = RoutedExperts(self, w, p, e) if e else None
        if L.experts:
            L.experts.layer = i
        if L.ff:
            up = self.mat(w, p + "ffn_up.weight")
            L.gate_up = DenseLinear(up if c.ffn_act == "gelu_up" else torch.cat([self.mat(w, p + "ffn_gate.weight"), up]))
            L.down = DenseLinear(self.mat(w, p + "ffn_down.weight"))

    def build_layer(self, L, w, i: int):
        p = f"blk.{i}."
        self.build_parts(L, w, i)
        L.attn_norm, L.post_attn_norm = self.vec(w, p + "attn_norm.weight"), self.vec(w, p + "post_attention_norm.weight")
        if L.ff or L.experts:
            L.ffn_norm, L.post_ffn_norm = self.vec(w, p + "ffn_norm.weight"), self.vec(w, p + "post_ffw_norm.weight")
        return L

    def nbytes(self, layers) -> int:
        n = self.loop_in.nbytes() if self.loop_in else 0
        for L in layers:
            n += L.mix.nbytes() + (L.experts.nbytes() if L.experts else 0) + (L.gate_up.nbytes() + L.down.nbytes() if L.ff else 0)
        return n

    def alloc_workspace(self, T: int, layers) -> None:
        c, cols = self.cfg, {"act": max(L.ff for L in layers), "gu": 2 * max(L.ff for L in layers)}
        for L in layers:
            for name, n in L.mix.workspace().items():
                cols[name] = max(cols.get(name, 0), n)
        self._ws = {k: torch.empty(T * max(1, n) * self.dtype.itemsize, dtype=torch.uint8, device=self.device) for k, n in cols.items()}
        e = lambda *s: torch.empty(*s, dtype=self.dtype, device=self.device)
        self.xn, self.y = e(T, c.d_model), e(T, c.d_model)
        self.cat = e(T, 2 * c.d_model) if c.loop else None             # [hidden | embedding], input of the loop projection
        parts = 0 if self.f32 or not self.has_latent else PART_FLOATS
        self.part_o = torch.empty(parts, dtype=torch.float32, device=self.device)
        self.part_ml = torch.empty(parts // 4, dtype=torch.float32, device=self.device)

    def ws(self, name: str, T: int, cols: int, dtype: torch.dtype | None = None) -> torch.Tensor:
        """Rows of a workspace in the activation type, or in another one (float rows of a decode step, which has few)."""
        return self._ws[name].view(dtype or self.dtype)[:T * cols].view(T, cols)

    # -- one forward call ------------------------------------------------------------------------------------
    def run(self, fb, kv, h: torch.Tensor, layers, after_layer) -> None:
        """The layer runs on the residual stream ``h``."""
        plan = self.plan(fb, h.shape[0], layers)
        first = layers[self.runs[0][0]].attn_norm
        self.embed_tokens(fb.tokens, h, None if self.runs[0][1] else first)
        n_pass = 0
        for r, (i, starts_pass) in enumerate(self.runs):
            L = layers[i]
            if starts_pass:
                self.enter_pass(h, L.attn_norm, n_pass)
                n_pass += 1
            nxt, to_pass = None, False
            if r + 1 < len(self.runs):
                to_pass = self.runs[r + 1][1]
                nxt = None if to_pass else layers[self.runs[r + 1][0]].attn_norm
            self.layer(L, h, fb, plan, kv, r, nxt, to_pass)
            after_layer(r, h)

    def plan(self, fb, T: int, layers) -> StackPlan:
        from ..ops import dense as ops
        angles = []
        for rot, f in zip(self.rotaries, self.freqs):
            a = torch.empty(T, f.numel(), 2, dtype=torch.float32, device=self.device)
            ops.rope_angles(fb.positions, f, rot.magnitude, a)
            angles.append(a)
        plan = StackPlan(angles)
        if self.has_latent:
            plan.latent = LatentPlan.build(fb, T, all(L.mix.chunk_fits for L in layers if isinstance(L.mix, LatentMixer)), self.device)
        if self.has_linear and not self.f32 and not fb.is_decode and self.linear_tc and fb.max_q_len > SHORT_ROWS:
            from ..ops import mixers as mixer_ops
            plan.chunks = mixer_ops.chunk_tables(fb.host_cu if fb.host_cu is not None else fb.cu_q.tolist(), self.device)
        return plan

    def mix(self, L, xn: torch.Tensor, fb, plan: StackPlan, kv, run: int) -> torch.Tensor:
        """A layer run's mixer up to its output product."""
        at = self.kv_index[run]
        return L.mix(xn, fb, plan, kv, kv.layers[at] if at is not None else None)

    def embed_tokens(self, tokens: torch.Tensor, h: torch.Tensor, first_norm: torch.Tensor | None) -> None:
        """h = the (normed) embedding; ``first_norm``: the first layer's input norm (None: a loop pass comes first)."""
        from ..ops import dense as ops
        T, d = h.shape
        cat = self.cat[:T] if self.cat is not None else None
        ops.resid_norm(h, self.embed, self.embed_norm, add=False, y_rows=tokens, w_next=first_norm, factor=self.cfg.embed_scale,
                       xn=self.xn[:T] if first_norm is not None else None, copy0=cat[:, d:] if cat is not None else None,
                       copy1=cat[:, :d] if cat is not None and first_norm is None else None, eps=self.cfg.rms_eps)

    def enter_pass(self, h: torch.Tensor, norm: torch.Tensor, n_pass: int) -> None:
        """h = Wloop [h | embedding] (+ the pass's vector); xn = norm(h).  The left half was written with the residual update before it."""
        from ..ops import dense as ops
        T, d = h.shape
        self.loop_in(self.cat[:T], h)
        step = self.loop_step[n_pass].expand(T, d) if self.loop_step is not None else None
        ops.resid_norm(h, step, w_next=norm, xn=self.xn[:T], eps=self.cfg.rms_eps)

    def _join(self, h: torch.Tensor, y, w_post: torch.Tensor, w_next: torch.Tensor | None, to_pass: bool, y_rows=None, y_w=None) -> None:
        """h += norm(y), and what the step behind it reads."""
        from ..ops import dense as ops
        T, d = h.shape
        ops.resid_norm(h, y, w_post, w_next=w_next, xn=self.xn[:T] if w_next is not None else None,
                       copy0=self.cat[:T, :d] if to_pass else None, eps=self.cfg.rms_eps, y_rows=y_rows, y_w=y_w)

    def layer(self, L, h: torch.Tensor, fb, plan: StackPlan, kv, run: int, next_norm: torch.Tensor | None, to_pass: bool) -> None:
        """xn holds the normed input; ``next_norm``: input norm of the layer that follows (None: a loop pass, or the end)."""
        T = h.shape[0]
        xn, y = self.xn[:T], self.y[:T]
        L.mix.wo(self.mix(L, xn, fb, plan, kv, run), y)
        if not L.ff and L.experts is None:
            self._join(h, y, L.post_attn_norm, next_norm, to_pass)
            return
        self._join(h, y, L.post_attn_norm, L.ffn_norm, False)
        if L.experts is not None:
            parts, rows, weights = L.experts(xn)
            self._join(h, parts, L.post_ffn_norm, next_norm, to_pass, rows, weights)
            return
        L.down(L.gate_up.activated(xn, self.ws("act", T, L.ff), self.ws("gu", T, 2 * L.ff), self.act), y)
        self._join(h, y, L.post_ffn_norm, next_norm, to_pass)

    def record_routing(self, experts: RoutedExperts, ids: torch.Tensor) -> None:
        """Router statistics (models/expert_placement.py); eager steps only."""
        stats = getattr(self.model, "expert_stats", None)
        if stats is not None and not torch.cuda.is_current_stream_capturing():
            stats.record(experts.layer, ids)

    def final_logits(self, rows: torch.Tensor, norm: torch.Tensor, head: DenseLinear, out: torch.Tensor) -> torch.Tensor:
        from ..ops import dense as ops
        xn = torch.empty(rows.shape, dtype=self.dtype, device=self.device)
        ops.resid_norm(rows, w_next=norm, xn=xn, eps=self.cfg.rms_eps)
        return head(xn, out)
