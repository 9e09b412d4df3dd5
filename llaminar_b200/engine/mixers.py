"""Decoder layers with a mixer of their own on the GPU (matrix LSTM; windowed attention beside retention): weights, workspace and the
kernel sequence of `CudaModel` for such models.

Per layer (the residual stream h is fp32; x is its copy in the activation type, bf16, or float in 32-bit mode):

    mLSTM      [q | k | v | g] = W x, gates = Wif x             linear_rows (decode) or linear_chunk
    parallel   [q | k | g | q' | k' | v' | g'] = W x            attn_prep, attention; linear_rows or linear_chunk
    y = Wo o (both sides)
    h += gain * norm(y) ; x = h                                 resid_norm (half the sum of both sides' norms first)
    h += gain * norm(Wd relu(Wu x)^2) ; x = h
    h += gain * norm(Wp (gelu(Wg x) * e)) ; x = h               e: this layer's columns of the token's side embedding

Decode steps keep the projections in front of a mixer in float.  Head sizes are zero-padded when the weights are loaded: to 64 or
128 in front of the tensor-core attention, to multiples of 8 in front of a recurrence.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..models.config import MatrixLSTM, ParallelMixers, Retention, WindowAttention
from ..models.mixers import mixer_kv_shapes, mixer_state_shapes, pad_to_multiple
from .dense import DenseLinear, pad8, pad_to


SHORT_ROWS = 4              # batches of portions up to this long advance the recurrences row by row


def _pad_heads(w: torch.Tensor, heads: int, size: int) -> torch.Tensor:
    """Rows of a projection [heads * n, k] -> [heads * size, k]."""
    k = w.shape[1]
    return pad_to(w.view(heads, -1, k), heads, size, k).view(-1, k)


def _pad_columns(w: torch.Tensor, heads: int, size: int) -> torch.Tensor:
    return pad_to(w.view(w.shape[0], heads, -1), w.shape[0], heads, size).view(w.shape[0], -1)


def _pad_gain(w: torch.Tensor, heads: int, size: int) -> torch.Tensor:
    return pad_to(w.view(heads, -1), heads, size).reshape(-1).contiguous()


@dataclass
class MixerPlan:
    """What the layers of one forward call share."""
    angles: list[torch.Tensor]          # per distinct rotation: [T, dims/2, 2]
    rows: torch.dtype                   # type of the projected rows in front of the mixers
    chunks: tuple | None = None         # how the chunk kernels cut the batch (None: row after row)


class MixerStack:
    def __init__(self, model, weights):
        c = self.cfg = model.cfg
        self.device, self.dtype = model.device, model.dtype
        self.f32 = self.dtype == torch.float32
        self.attn_tc = self.linear_tc = True            # tcgen05 forms of the prompt kernels where the sizes fit
        # sums stay in 32 bits: no TF32 operands in 32-bit mode, no 16-bit reduction of split products otherwise
        if self.f32:
            torch.backends.cuda.matmul.allow_tf32 = False
        else:
            torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        self.embed = self._mat(weights, "token_embd.weight")
        self.side = self._mat(weights, "side_embd.weight") if c.side_dim else None
        self.kv_layer_shapes = mixer_kv_shapes(c, self.head_pad)
        self.state_shapes = mixer_state_shapes(c, 8)
        self.n_kv_layers = len(self.kv_layer_shapes)
        from .. import ops
        self.scratch = ops.scratch_for(self.device)
        self.status = self.scratch.status                               # word that a kernel sets when a bounded wait runs out
        self.rotaries: list = []
        self.freqs: list[torch.Tensor] = []
        self._kv_i = self._state_i = 0

    def head_pad(self, dim: int) -> int:
        """Head size of the attention kernels for heads of ``dim`` values."""
        from ..ops import grouped as ops
        if self.f32 or dim > max(ops.HEAD_SIZES):
            return pad8(dim)
        return min(s for s in ops.HEAD_SIZES if s >= dim)

    def _mat(self, w, name: str) -> torch.Tensor:
        return w[name].to_float().to(self.device).to(self.dtype)

    def head_matrix(self, w) -> torch.Tensor:
        return self._mat(w, "output.weight")

    def _vec(self, w, name: str) -> torch.Tensor:
        return w[name].to_float().to(device=self.device, dtype=torch.float32).contiguous()

    # -- weights ---------------------------------------------------------------------------------------------
    def build_layer(self, L, w, i: int):
        c, m, p = self.cfg, self.cfg.mixers[i], f"blk.{i}."
        L.index, L.mixer = i, m
        gain = lambda name: (self._vec(w, p + name + "_norm.weight") * self._vec(w, p + name + "_scale.weight") * c.residual_mult).contiguous()
        L.post_mix = gain("post_attention")
        if isinstance(m, MatrixLSTM):
            L.left, L.right = None, self._build_lstm(w, p, m)
            gates = torch.cat([self._mat(w, p + "lstm_i.weight"), self._mat(w, p + "lstm_f.weight")])
            L.gate_proj, L.gate_col = DenseLinear(gates), L.right.cols
            # decode steps (float rows) take the gates from the one product
            L.proj = DenseLinear(torch.cat(L.right.rows + [pad_to(gates, pad8(gates.shape[0]), gates.shape[1])]))
        else:
            L.left, L.right = self._build_attention(w, p, m.left), self._build_retention(w, p, m.right)
            L.right.offs = [x + L.left.cols for x in L.right.offs]
            L.proj = DenseLinear(torch.cat(L.left.rows + L.right.rows))
            L.left_out, L.right_out = self._vec(w, p + "attn_out_norm.weight"), self._vec(w, p + "ret_out_norm.weight")
        for part in (L.left, L.right):
            if part is not None:
                del part.rows
        L.ff = c.ff_width(i)
        if L.ff:
            L.post_ffn = gain("post_ffw")
            L.up, L.down = DenseLinear(self._mat(w, p + "ffn_up.weight")), DenseLinear(self._mat(w, p + "ffn_down.weight"))
        if c.side_dim:
            n = pad8(c.side_dim)
            g, pr = self._mat(w, p + "side_gate.weight"), self._mat(w, p + "side_proj.weight")
            L.side_gate, L.side_proj = DenseLinear(pad_to(g, n, g.shape[1])), DenseLinear(pad_to(pr, pr.shape[0], n))
            L.side_norm = (self._vec(w, p + "side_norm.weight") * c.residual_mult).contiguous()
        return L

    def _part(self, m, rows: list[torch.Tensor], offs_of: list[int]):
        """A mixer's projections: stacked rows and the first column of each in the product."""
        part = type("Part", (), {})()
        part.m, part.rows, part.offs, at = m, rows, [], 0
        for r in rows:
            part.offs.append(at)
            at += r.shape[0]
        part.cols = at
        return part

    def _build_attention(self, w, p: str, m: WindowAttention):
        d = self.head_pad(m.dim)
        q, k, g = (_pad_heads(self._mat(w, p + n + ".weight"), h, d) for n, h in (("attn_q", m.heads), ("attn_k", m.kv_heads), ("attn_gate", m.heads)))
        part = self._part(m, [q, k, g], [])
        part.dim, part.kv = d, self._kv_i
        self._kv_i += 1
        part.q_norm, part.k_norm = _pad_gain(self._vec(w, p + "attn_q_norm.weight"), m.heads, d), _pad_gain(self._vec(w, p + "attn_k_norm.weight"), m.kv_heads, d)
        part.sink = self._vec(w, p + "attn_sinks.weight") if m.sinks else None
        part.wo = DenseLinear(_pad_columns(self._mat(w, p + "attn_output.weight"), m.heads, d))
        return part

    def _build_linear(self, w, p: str, m):
        d, v = pad8(m.dim), pad8(m.vdim)
        rows = [_pad_heads(self._mat(w, f"{p}{n}.weight"), m.heads, s) for n, s in (("q", d), ("k", d), ("v", v), ("g", v))]
        part = self._part(m, rows, [])
        part.dim, part.vdim, part.state = d, v, self._state_i
        self._state_i += 1
        part.wo = DenseLinear(_pad_columns(self._mat(w, p + "output.weight"), m.heads, v))
        part.norm = part.gates = part.decay = part.rot = None
        part.q_scale = part.k_scale = 1.0
        return part

    def _build_lstm(self, w, p: str, m: MatrixLSTM):
        part = self._build_linear(w, p + "lstm_", m)
        part.norm = _pad_gain(self._vec(w, p + "lstm_norm.weight"), m.heads, part.vdim)
        part.gates = (self._vec(w, p + "lstm_i.bias"), self._vec(w, p + "lstm_f.bias"), m.gate_cap)
        part.q_scale = m.dim ** -0.5
        return part

    def _build_retention(self, w, p: str, m: Retention):
        part = self._build_linear(w, p + "ret_", m)
        part.decay = torch.tensor(m.decay, dtype=torch.float32, device=self.device)
        part.k_scale = m.dim ** -0.5
        if m.rotary not in self.rotaries:
            self.rotaries.append(m.rotary)
            self.freqs.append(torch.tensor(m.rotary.frequencies(), dtype=torch.float64, device=self.device))
        part.rot = self.rotaries.index(m.rotary)
        return part

    def _linears(self, L) -> list[DenseLinear]:
        out = [L.proj, L.right.wo]
        if isinstance(L.mixer, MatrixLSTM):
            out.append(L.gate_proj)
        else:
            out.append(L.left.wo)
        if L.ff:
            out += [L.up, L.down]
        if self.cfg.side_dim:
            out += [L.side_gate, L.side_proj]
        return out

    def nbytes(self, layers) -> int:
        return sum(x.nbytes() for L in layers for x in self._linears(L))

    def alloc_workspace(self, T: int, layers) -> None:
        c = self.cfg
        e = lambda n, dt=self.dtype: torch.empty(T * max(1, n), dtype=dt, device=self.device)
        attn = [L.left.m.heads * L.left.dim for L in layers if L.left is not None]
        lin = [L.right.m.heads * L.right.vdim for L in layers]
        self._ws = {"q": e(max(attn, default=0)), "oa": e(max(attn, default=0)), "ol": e(max(lin)),
                    "act": e(max(max(L.ff for L in layers), pad8(c.side_dim))), "raw": e(max(max(L.ff for L in layers), pad8(c.side_dim), max(lin)))}
        # projected rows: float in a decode step (few rows) and in 32-bit mode, the activation type in prompts; one buffer for both
        self._rows = torch.empty(T * max(L.proj.n_out for L in layers) * (4 if self.f32 else 2), dtype=torch.uint8, device=self.device)
        self._gates = torch.empty(T * 2 * max((L.mixer.heads for L in layers if isinstance(L.mixer, MatrixLSTM)), default=1), dtype=torch.float32, device=self.device)
        self.x, self.y, self.y2 = (torch.empty(T, c.d_model, dtype=self.dtype, device=self.device) for _ in range(3))

    def ws(self, name: str, T: int, cols: int) -> torch.Tensor:
        return self._ws[name][:T * cols].view(T, cols)

    # -- one forward call ------------------------------------------------------------------------------------
    def run(self, fb, kv, h: torch.Tensor, layers, after_layer) -> None:
        """The layers on the residual stream ``h``."""
        from ..ops import dense as ops
        c, T = self.cfg, h.shape[0]
        plan = self.plan(fb, T)
        ops.resid_norm(h, self.embed, None, add=False, y_rows=fb.tokens, factor=c.embed_scale, copy0=self.x[:T], eps=c.rms_eps)
        for L in layers:
            self.layer(L, h, fb, plan, kv)
            after_layer(L.index, h)

    def plan(self, fb, T: int) -> MixerPlan:
        from ..ops import dense as ops
        from ..ops import mixers as mixer_ops
        angles = []
        for rot, f in zip(self.rotaries, self.freqs):
            a = torch.empty(T, f.numel(), 2, dtype=torch.float32, device=self.device)
            ops.rope_angles(fb.positions, f, rot.magnitude, a)
            angles.append(a)
        plan = MixerPlan(angles, torch.float32 if self.f32 or fb.is_decode else self.dtype)
        if not self.f32 and not fb.is_decode and self.linear_tc and fb.max_q_len > SHORT_ROWS:
            plan.chunks = mixer_ops.chunk_tables(fb.host_cu if fb.host_cu is not None else fb.cu_q.tolist(), self.device)
        return plan

    def layer(self, L, h: torch.Tensor, fb, plan: MixerPlan, kv) -> None:
        """x holds the layer's input in the activation type, and its output's at the end."""
        from ..ops import dense as ops
        c, T = self.cfg, h.shape[0]
        x, y, eps = self.x[:T], self.y[:T], c.rms_eps
        rows = self._rows.view(plan.rows)[:T * L.proj.n_out].view(T, L.proj.n_out)
        L.proj(x, rows)
        if L.left is None:
            n = L.gate_proj.n_out
            gates = rows[:, L.gate_col:L.gate_col + n] if rows.dtype == torch.float32 else L.gate_proj(x, self._gates[:T * n].view(T, n))
            L.right.wo(self._linear(L.right, rows, gates, fb, plan, kv), y)
            ops.resid_norm(h, y, L.post_mix, copy0=x, center_post=True, eps=eps)
        else:
            y2 = self.y2[:T]
            L.left.wo(self._attention(L.left, rows, fb, plan, kv), y)
            L.right.wo(self._linear(L.right, rows, None, fb, plan, kv), y2)
            ops.resid_norm(h, y, L.post_mix, y2=y2, w_y=L.left_out, w_y2=L.right_out, copy0=x, center_post=True, eps=eps)
        if L.ff:
            L.down(L.up.activated(x, self.ws("act", T, L.ff), self.ws("raw", T, L.ff), ops.ACT_RELU2), y)
            ops.resid_norm(h, y, L.post_ffn, copy0=x, center_post=True, eps=eps)
        if c.side_dim:
            n = L.side_gate.n_out
            side = (self.side, L.index * c.side_dim, c.side_dim, fb.tokens)
            L.side_proj(L.side_gate.activated(x, self.ws("act", T, n), self.ws("raw", T, n), ops.ACT_GELU_SIDE, side), y)
            ops.resid_norm(h, y, L.side_norm, copy0=x, eps=eps)

    def _attention(self, P, rows: torch.Tensor, fb, plan: MixerPlan, kv) -> torch.Tensor:
        from ..ops import grouped as ops
        m, T = P.m, rows.shape[0]
        kvl, H, D = kv.layers[P.kv], m.heads, P.dim
        q, o = self.ws("q", T, H * D).view(T, H, D), self.ws("oa", T, H * D)
        ops.attn_prep(rows, P.offs[0], P.offs[1], P.offs[1], P.q_norm, P.k_norm, fb.positions, fb.seq_ids, fb.block_table, q, kvl, m.dim, self.cfg.rms_eps)
        gate = rows[:, P.offs[2]:P.offs[2] + H * D]
        fits = not self.f32 and D in ops.HEAD_SIZES
        if fits and fb.is_decode and H // m.kv_heads <= ops.DECODE_GROUP:
            splits = ops.decode_splits(T, m.kv_heads, D, fb.block_table.shape[1], m.window, self.scratch)
            ops.attn_decode(q, kvl, o, fb.block_table, fb.seq_lens, m.scale, splits, m.window, P.sink, gate, self.scratch)
        elif fits and not fb.is_decode:
            tc = self.attn_tc and ops.prefill_tc(D, fb.max_q_len)
            ops.attn_prefill(q, kvl, o, fb.block_table, fb.cu_q, fb.ctx_lens, m.scale, fb.max_q_len, m.window, P.sink, gate, self.status if tc else None)
        else:
            ops.attn_plain(q, kvl, o, fb.positions, fb.seq_ids, fb.block_table, m.window, m.scale, P.sink, gate)
        return o

    def _linear(self, P, rows: torch.Tensor, gates, fb, plan: MixerPlan, kv) -> torch.Tensor:
        from ..ops import mixers as ops
        m, T = P.m, rows.shape[0]
        o = self.ws("ol", T, m.heads * P.vdim)
        state = kv.hybrid.layers[P.state]
        args = (rows, P.offs, (gates, *P.gates) if gates is not None else None, P.decay, plan.angles[P.rot] if P.rot is not None else None, P.q_scale, P.k_scale)
        args += (None if fb.is_decode else fb.cu_q, fb.positions, fb.state_slots, state, m.vdim, P.norm, gates is None, o, self.cfg.rms_eps)
        if plan.chunks is not None and ops.linear_chunk_fits(P.dim, P.vdim):
            ops.linear_chunk(*args, plan.chunks, self.ws("raw", T, m.heads * P.vdim), self.status)
        else:
            ops.linear_rows(*args)
        return o

    def final_logits(self, rows: torch.Tensor, norm: torch.Tensor, head: DenseLinear, out: torch.Tensor) -> torch.Tensor:
        from ..ops import dense as ops
        xn = torch.empty(rows.shape, dtype=self.dtype, device=self.device)
        ops.resid_norm(rows, w_next=norm, xn=xn, center_next=True, eps=self.cfg.rms_eps)
        return head(xn, out)
