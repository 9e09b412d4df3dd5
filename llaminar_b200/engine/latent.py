"""Latent-attention decoder layers on the GPU: weights, workspace and the kernel sequence of `CudaModel` for such models.

Per layer (the residual stream h is fp32, everything else bf16, or float in 32-bit mode):

    [q latent | kv latent | rotated key part] = Wdown xn        one product
    norms of both latents, rotation, cache append               latent_prep
    q = Wuq cq
    attention                                                   latent_rows (queries moved into the latent space: decode steps and
                                                                short portions) or latent_chunk (keys and values written out)
    y = Wo o ; h += norm(y) ; xn = norm(h)                      resid_norm
    act = gelu(Wg xn) * (Wu xn) ; y = Wd act                    fused into the product up to eight rows
    h += norm(y) ; xn = norm(h) of the next layer               resid_norm

Matrix products run on `gemv_dense` up to eight rows and on cuBLAS above.  Head sizes and the latent are zero-padded to
multiples of 8 values when the weights are loaded, so that every row the kernels copy starts on a 16-byte boundary.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ..models.config import LatentAttention
from .dense import DenseLinear, pad8, pad_to

SHORT_ROWS = 8                 # portions of up to this many tokens attend row by row in the latent space
PART_FLOATS = 1 << 23          # scratch of the split row kernel
PLAIN_ROWS = 1024              # rows per launch where the row kernel serves whole prompts (32-bit mode, unusual sizes)


@dataclass(frozen=True)
class PaddedSizes:
    """A mixer's sizes as the kernels see them."""
    heads: int
    dim: int
    rot: int
    vdim: int
    q_rank: int
    latent: int
    width: int

    @staticmethod
    def of(m: LatentAttention) -> "PaddedSizes":
        return PaddedSizes(m.heads, pad8(m.dim), pad8(m.rot_dim), pad8(m.vdim), pad8(m.q_rank), pad8(m.kv_rank), m.cache_width)


@dataclass
class BatchPlan:
    """How one forward call's rows attend; the same for every layer of equal sizes and window."""
    angles: list[torch.Tensor]                       # per distinct rotation: [T, dims/2, 2]
    rows: torch.Tensor | None = None                 # tokens of the short portions (None: every row of the batch)
    n_rows: int = 0
    long: list[tuple[int, int, int, int]] = field(default_factory=list)      # (sequence, first row, rows, context)
    keys: dict = field(default_factory=dict)         # window -> (sequence table on the device, keys in all, longest, longest query)
    max_keys: int = 0


class LatentStack:
    """Everything of `CudaModel` that is specific to latent-attention models."""

    def __init__(self, model, weights):
        c = self.cfg = model.cfg
        self.device, self.dtype = model.device, model.dtype
        self.f32 = self.dtype == torch.float32
        self.rows_tc = self.chunk_tc = True             # tcgen05 forms of the attention kernels where the sizes fit
        # sums stay in 32 bits: no TF32 operands in 32-bit mode, no 16-bit reduction of split products otherwise
        if self.f32:
            torch.backends.cuda.matmul.allow_tf32 = False
        else:
            torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        self.embed = self._mat(weights, "token_embd.weight")
        self.embed_norm = self._vec(weights, "token_embd_norm.weight")
        self.loop_in = DenseLinear(self._mat(weights, "loop_in.weight")) if c.loop else None
        from .. import ops
        self.status = ops.scratch_for(self.device).status               # word that a kernel sets when a bounded wait runs out
        self.runs = c.layer_runs()                       # looped layers have a cache layer per pass, each with its own row width
        self.kv_row_widths = [c.mixers[i].cache_width for i, _ in self.runs]
        self.kv_head_shapes = self.state_shapes = None
        self.n_kv_layers = len(self.runs)
        self.rotaries: list = []
        self.freqs: list[torch.Tensor] = []

    def _mat(self, w, name: str) -> torch.Tensor:
        return w[name].to_float().to(self.device).to(self.dtype)

    def _vec(self, w, name: str) -> torch.Tensor:
        return w[name].to_float().to(device=self.device, dtype=torch.float32).contiguous()

    # -- weights ---------------------------------------------------------------------------------------------
    def build_layer(self, L, w, i: int):
        from ..ops import latent as ops
        c, m, p = self.cfg, self.cfg.mixers[i], f"blk.{i}."
        s = PaddedSizes.of(m)
        L.index, L.mixer, L.sizes = i, m, s
        L.attn_norm, L.post_attn_norm = self._vec(w, p + "attn_norm.weight"), self._vec(w, p + "post_attention_norm.weight")
        L.q_a_norm, L.kv_a_norm = self._vec(w, p + "attn_q_a_norm.weight"), self._vec(w, p + "attn_kv_a_norm.weight")
        L.sink = self._vec(w, p + "attn_sinks.weight") if m.sinks else None
        L.down_a = DenseLinear(torch.cat([self._mat(w, p + "attn_q_a.weight"), self._mat(w, p + "attn_kv_a.weight")]))
        q = self._mat(w, p + "attn_q_b.weight").view(m.heads, m.dim + m.rot_dim, m.q_rank)
        q = torch.cat([pad_to(q[:, :m.dim], s.heads, s.dim, s.q_rank), pad_to(q[:, m.dim:], s.heads, s.rot, s.q_rank)], dim=1)
        L.q_b = DenseLinear(q.reshape(-1, s.q_rank))
        k = pad_to(self._mat(w, p + "attn_k_b.weight").view(m.heads, m.dim, m.kv_rank), s.heads, s.dim, s.latent)
        v = pad_to(self._mat(w, p + "attn_v_b.weight").view(m.heads, m.vdim, m.kv_rank), s.heads, s.vdim, s.latent)
        L.k_b, L.v_b = k, v                                             # [heads, dim, latent], [heads, vdim, latent]
        L.k_bt = k.transpose(1, 2).contiguous()                         # [heads, latent, dim]: rows of the small-batch product
        o = self._mat(w, p + "attn_output.weight").view(-1, m.heads, m.vdim)
        L.wo = DenseLinear(pad_to(o, o.shape[0], s.heads, s.vdim).view(o.shape[0], -1))
        if m.rotary not in self.rotaries:
            self.rotaries.append(m.rotary)
            self.freqs.append(torch.tensor(m.rotary.frequencies(), dtype=torch.float64, device=self.device))
        L.chunk_tc = not self.f32 and ops.chunk_tc_fits(s.dim, s.rot, s.vdim)
        L.rot_index = self.rotaries.index(m.rotary)
        L.ff = c.ff_width(i)
        if L.ff:
            L.ffn_norm, L.post_ffn_norm = self._vec(w, p + "ffn_norm.weight"), self._vec(w, p + "post_ffw_norm.weight")
            L.gate_up = DenseLinear(torch.cat([self._mat(w, p + "ffn_gate.weight"), self._mat(w, p + "ffn_up.weight")]), gelu_pair=True)
            L.down = DenseLinear(self._mat(w, p + "ffn_down.weight"))
        return L

    def nbytes(self, layers) -> int:
        n = (self.loop_in.nbytes() if self.loop_in else 0)
        for L in layers:
            n += sum(x.nbytes() for x in (L.down_a, L.q_b, L.wo))
            n += (2 * L.k_b.numel() + L.v_b.numel()) * L.k_b.element_size()
            if L.ff:
                n += L.gate_up.nbytes() + L.down.nbytes()
        return n

    def alloc_workspace(self, T: int, layers) -> None:
        c = self.cfg
        cols = {"down": lambda L: L.down_a.n_out, "cq": lambda L: L.sizes.q_rank, "q": lambda L: L.q_b.n_out, "o": lambda L: L.wo.k,
                "act": lambda L: L.ff, "gu": lambda L: 2 * L.ff}
        self._ws = {k: torch.empty(T * max(1, max(f(L) for L in layers)), dtype=self.dtype, device=self.device) for k, f in cols.items()}
        e = lambda *s: torch.empty(*s, dtype=self.dtype, device=self.device)
        self.xn, self.y = e(T, c.d_model), e(T, c.d_model)
        self.cat = e(T, 2 * c.d_model) if c.loop else None             # [hidden | embedding], input of the loop projection
        self.part_o = torch.empty(0 if self.f32 else PART_FLOATS, dtype=torch.float32, device=self.device)
        self.part_ml = torch.empty(0 if self.f32 else PART_FLOATS // 4, dtype=torch.float32, device=self.device)

    def ws(self, name: str, T: int, cols: int) -> torch.Tensor:
        return self._ws[name][:T * cols].view(T, cols)

    # -- one forward call ------------------------------------------------------------------------------------
    def run(self, fb, kv, h: torch.Tensor, layers, after_layer) -> None:
        """The layer runs on the residual stream ``h``."""
        bp = self.plan(fb, h.shape[0], layers)
        first = layers[self.runs[0][0]].attn_norm
        self.embed_tokens(fb.tokens, h, None if self.runs[0][1] else first)
        for r, (i, starts_pass) in enumerate(self.runs):
            L = layers[i]
            if starts_pass:
                self.enter_pass(h, L.attn_norm)
            nxt, to_pass = None, False
            if r + 1 < len(self.runs):
                to_pass = self.runs[r + 1][1]
                nxt = None if to_pass else layers[self.runs[r + 1][0]].attn_norm
            self.layer(L, h, fb, bp, kv.layers[r], nxt, to_pass)
            after_layer(r, h)

    def plan(self, fb, T: int, layers) -> BatchPlan:
        from ..ops import latent as ops
        angles = []
        for rot, f in zip(self.rotaries, self.freqs):
            a = torch.empty(T, f.numel(), 2, dtype=torch.float32, device=self.device)
            ops.rope_angles(fb.positions, f, rot.magnitude, a)
            angles.append(a)
        bp = BatchPlan(angles, n_rows=T, max_keys=fb.block_table.shape[1] * 64)
        if fb.is_decode or self.f32 or not all(self._chunk_fits(L) for L in layers):
            return bp
        cu = fb.host_cu if fb.host_cu is not None else fb.cu_q.tolist()
        ctx = fb.host_ctx if fb.host_ctx is not None else fb.ctx_lens.tolist()
        short = []
        for b, n0 in enumerate(ctx):
            n = cu[b + 1] - cu[b]
            if n > SHORT_ROWS:
                bp.long.append((b, cu[b], n, n0))
            else:
                short.extend(range(cu[b], cu[b + 1]))
        if bp.long:
            bp.n_rows = len(short)
            bp.rows = torch.tensor(short, dtype=torch.int32, device=self.device) if short else None
        return bp

    @staticmethod
    def _chunk_fits(L) -> bool:
        from ..ops import latent as ops
        return ops.chunk_has_kernel(L.sizes.dim + L.sizes.rot, L.sizes.vdim)

    def embed_tokens(self, tokens: torch.Tensor, h: torch.Tensor, first_norm: torch.Tensor | None) -> None:
        """h = norm(embedding); ``first_norm``: the first layer's input norm (None: a loop pass comes first)."""
        from ..ops import latent as ops
        T, d = h.shape
        cat = self.cat[:T] if self.cat is not None else None
        ops.resid_norm(h, self.embed, self.embed_norm, add=False, y_rows=tokens, w_next=first_norm,
                       xn=self.xn[:T] if first_norm is not None else None, copy0=cat[:, d:] if cat is not None else None,
                       copy1=cat[:, :d] if cat is not None and first_norm is None else None, eps=self.cfg.rms_eps)

    def enter_pass(self, h: torch.Tensor, norm: torch.Tensor) -> None:
        """h = Wloop [h | embedding]; xn = norm(h).  The left half was written with the residual update before it."""
        from ..ops import latent as ops
        T = h.shape[0]
        self.loop_in(self.cat[:T], h)
        ops.resid_norm(h, w_next=norm, xn=self.xn[:T], eps=self.cfg.rms_eps)

    def _join(self, h: torch.Tensor, w_post: torch.Tensor, w_next: torch.Tensor | None, to_pass: bool) -> None:
        """h += norm(y), and what the step behind it reads."""
        from ..ops import latent as ops
        T, d = h.shape
        ops.resid_norm(h, self.y[:T], w_post, w_next=w_next, xn=self.xn[:T] if w_next is not None else None,
                       copy0=self.cat[:T, :d] if to_pass else None, eps=self.cfg.rms_eps)

    def layer(self, L, h: torch.Tensor, fb, bp: BatchPlan, kv_layer: torch.Tensor, next_norm: torch.Tensor | None, to_pass: bool) -> None:
        """xn holds the normed input; ``next_norm``: input norm of the layer that follows (None: a loop pass, or the end)."""
        from ..ops import latent as ops
        c, m, s = self.cfg, L.mixer, L.sizes
        T = h.shape[0]
        down = L.down_a(self.xn[:T], self.ws("down", T, L.down_a.n_out))
        cq = self.ws("cq", T, s.q_rank)
        ops.latent_prep(down, L.q_a_norm, L.kv_a_norm, bp.angles[L.rot_index], fb.positions, fb.seq_ids, fb.block_table, cq, kv_layer,
                        m.rot_dim, s.latent, c.rms_eps)
        q = L.q_b(cq, self.ws("q", T, L.q_b.n_out)).view(T, s.heads, s.dim + s.rot)
        o = self.ws("o", T, L.wo.k)
        if bp.n_rows:
            self._attend_rows(L, q, o.view(T, s.heads, s.vdim), fb, bp, kv_layer)
        if bp.long:
            self._attend_chunks(L, q, o, fb, bp, kv_layer)
        y = self.y[:T]
        L.wo(o, y)
        if not L.ff:
            self._join(h, L.post_attn_norm, next_norm, to_pass)
            return
        self._join(h, L.post_attn_norm, L.ffn_norm, False)
        L.down(L.gate_up.gelu(self.xn[:T], self.ws("act", T, L.ff), self.ws("gu", T, 2 * L.ff)), y)
        self._join(h, L.post_ffn_norm, next_norm, to_pass)

    def _attend_rows(self, L, q: torch.Tensor, o3: torch.Tensor, fb, bp: BatchPlan, kv_layer: torch.Tensor) -> None:
        s = L.sizes
        T = q.shape[0]
        n = bp.n_rows
        step = PLAIN_ROWS if bp.rows is None and n > PLAIN_ROWS else n
        for r0 in range(0, n, step):
            r1 = min(n, r0 + step)
            if bp.rows is not None:
                rows, qs, dst = bp.rows, q.index_select(0, bp.rows.long()), None
            elif step < n:
                rows, qs, dst = torch.arange(r0, r1, dtype=torch.int32, device=self.device), q[r0:r1], o3[r0:r1]
            else:
                rows, qs, dst = None, q, o3
            out = self._rows_values(L, q, qs[:, :, :s.dim].transpose(0, 1), rows, fb, bp, kv_layer, dst)
            if dst is None:
                o3[bp.rows.long()] = out.transpose(0, 1)

    def _rows_values(self, L, q, q_nope, rows, fb, bp: BatchPlan, kv_layer, dst):
        """Attention values [heads, rows, vdim] of single rows; ``dst`` [rows, heads, vdim] receives them when given."""
        from ..ops import latent as ops
        m, s = L.mixer, L.sizes
        n = q_nope.shape[1]
        e = lambda c: torch.empty(s.heads, n, c, dtype=self.dtype, device=self.device)
        q_lat, o_lat = e(s.latent), e(s.latent)
        if ops.gemv_fits(L.k_bt, q_nope):
            ops.gemv_dense(L.k_bt, q_nope, q_lat)
        else:
            torch.bmm(q_nope, L.k_b, out=q_lat)
        max_keys = min(bp.max_keys, m.window) if m.window else bp.max_keys
        group = ops.rows_group(kv_layer, s.latent, m.rot_dim, s.heads, self.rows_tc)
        splits = ops.rows_splits(n, s.heads, group, self.rows_tc, max_keys, s.latent, self.part_o.numel())
        ops.latent_rows(q_lat, q, s.dim, bp.angles[L.rot_index], rows, fb.positions, fb.seq_ids, fb.block_table, kv_layer, m.rot_dim, m.window,
                        m.scale, L.sink, o_lat, self.part_o, self.part_ml, splits, group, self.status)
        out = dst.transpose(0, 1) if dst is not None else e(s.vdim)
        if ops.gemv_fits(L.v_b, o_lat):
            ops.gemv_dense(L.v_b, o_lat, out)
        else:
            torch.bmm(o_lat, L.v_b.transpose(1, 2), out=out)
        return out

    def _chunk_keys(self, bp: BatchPlan, window: int):
        """Sequence table of the prompt chunks for a window: which keys each needs and where they land in the key buffer."""
        got = bp.keys.get(window)
        if got is None:
            table, off, longest, max_q = [], 0, 0, 0
            for b, q0, n, ctx in bp.long:
                k0 = max(0, ctx - window + 1) if window else 0
                kn = ctx + n - k0
                table.append((b, q0, n, ctx, off, k0, kn, 0))
                off, longest, max_q = off + pad8(kn), max(longest, kn), max(max_q, n)
            got = bp.keys[window] = (torch.tensor(table, dtype=torch.int32, device=self.device), off, longest, max_q)
        return got

    def _attend_chunks(self, L, q: torch.Tensor, o: torch.Tensor, fb, bp: BatchPlan, kv_layer: torch.Tensor) -> None:
        from ..ops import latent as ops
        m, s = L.mixer, L.sizes
        seqs, n_keys, longest, max_q = self._chunk_keys(bp, m.window)      # n_keys: with the rows up to the next multiple of 8
        lat = torch.empty(n_keys, s.width, dtype=self.dtype, device=self.device)
        ops.latent_gather(kv_layer, seqs, pad8(longest), fb.block_table, lat)
        c = lat[:, :s.latent]
        k = torch.mm(c, L.k_b.view(-1, s.latent).t())
        v_b = L.v_b.view(-1, s.latent)
        tc = L.chunk_tc and self.chunk_tc
        v = torch.mm(v_b, c.t()) if tc else torch.mm(c, v_b.t())
        ops.latent_chunk(q, bp.angles[L.rot_index], k, v, lat, s.latent, seqs, max_q, o, s.dim, s.rot, s.vdim, m.window, m.scale, L.sink,
                         self.status if tc else None)

    def final_logits(self, rows: torch.Tensor, norm: torch.Tensor, head: DenseLinear, out: torch.Tensor) -> torch.Tensor:
        from ..ops import latent as ops
        xn = torch.empty(rows.shape, dtype=self.dtype, device=self.device)
        ops.resid_norm(rows, w_next=norm, xn=xn, eps=self.cfg.rms_eps)
        return head(xn, out)
