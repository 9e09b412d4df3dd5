"""Latent attention on the GPU: a layer's weights and its kernel sequence between the input norm and the output product.

    [q latent | kv latent | rotated key part | gate] = Wdown xn     one product
    norms of both latents, rotation, cache append               latent_prep
    q = Wuq cq
    attention                                                   latent_rows (queries moved into the latent space: decode steps and
                                                                short portions) or latent_chunk (keys and values written out)

Head sizes and the latent are zero-padded to multiples of 8 values when the weights are loaded, so that every row the kernels copy
starts on a 16-byte boundary.  Rotated parts are stored in the order in which pair i is (i, i + half).
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
class LatentPlan:
    """How one forward call's rows attend; the same for every layer of equal sizes and window."""
    rows: torch.Tensor | None = None                 # tokens of the short portions (None: every row of the batch)
    n_rows: int = 0
    long: list[tuple[int, int, int, int]] = field(default_factory=list)      # (sequence, first row, rows, context)
    keys: dict = field(default_factory=dict)         # window -> (sequence table on the device, keys in all, longest, longest query)
    max_keys: int = 0

    @staticmethod
    def build(fb, T: int, chunks: bool, device) -> "LatentPlan":
        """``chunks``: portions may run on the chunk kernels."""
        plan = LatentPlan(n_rows=T, max_keys=fb.block_table.shape[1] * 64)
        if fb.is_decode or not chunks:
            return plan
        cu = fb.host_cu if fb.host_cu is not None else fb.cu_q.tolist()
        ctx = fb.host_ctx if fb.host_ctx is not None else fb.ctx_lens.tolist()
        short = []
        for b, n0 in enumerate(ctx):
            n = cu[b + 1] - cu[b]
            if n > SHORT_ROWS:
                plan.long.append((b, cu[b], n, n0))
            else:
                short.extend(range(cu[b], cu[b + 1]))
        if plan.long:
            plan.n_rows = len(short)
            plan.rows = torch.tensor(short, dtype=torch.int32, device=device) if short else None
        return plan


class LatentMixer:
    """One layer's latent attention.  ``stack``: the `AttentionStack` it belongs to (workspace, rotations, activation type)."""

    def __init__(self, stack, w, p: str, m: LatentAttention):
        from ..ops import latent as ops
        mat, s = lambda name: stack.mat(w, p + name), PaddedSizes.of(m)
        self.stack, self.m, self.sizes, self.device, self.dtype = stack, m, s, stack.device, stack.dtype
        order = m.rotary.halves_order(m.rot_dim)
        self.q_a_norm, self.kv_a_norm = stack.vec(w, p + "attn_q_a_norm.weight"), stack.vec(w, p + "attn_kv_a_norm.weight")
        self.sink = stack.vec(w, p + "attn_sinks.weight") if m.sinks else None
        kv_a = mat("attn_kv_a.weight")
        down = [mat("attn_q_a.weight"), kv_a[:m.kv_rank], kv_a[m.kv_rank:][order]]
        self.gate_col = 0
        if m.gated:                                                     # behind the rest, from a 16-byte boundary on
            n, d = m.q_rank + m.kv_rank + m.rot_dim, kv_a.shape[1]
            g = pad_to(mat("attn_gate.weight").view(m.heads, m.vdim, d), s.heads, s.vdim, d).view(-1, d)
            self.gate_col = pad8(n)
            down += [kv_a.new_zeros(self.gate_col - n, d), g]
        self.down = DenseLinear(torch.cat(down))
        q = mat("attn_q_b.weight").view(m.heads, m.dim + m.rot_dim, m.q_rank)
        q = torch.cat([pad_to(q[:, :m.dim], s.heads, s.dim, s.q_rank), pad_to(q[:, m.dim:][:, order], s.heads, s.rot, s.q_rank)], dim=1)
        self.q_b = DenseLinear(q.reshape(-1, s.q_rank))
        self.k_b = pad_to(mat("attn_k_b.weight").view(m.heads, m.dim, m.kv_rank), s.heads, s.dim, s.latent)         # [heads, dim, latent]
        self.v_b = pad_to(mat("attn_v_b.weight").view(m.heads, m.vdim, m.kv_rank), s.heads, s.vdim, s.latent)       # [heads, vdim, latent]
        self.k_bt = self.k_b.transpose(1, 2).contiguous()               # [heads, latent, dim]: rows of the small-batch product
        o = mat("attn_output.weight").view(-1, m.heads, m.vdim)
        self.wo = DenseLinear(pad_to(o, o.shape[0], s.heads, s.vdim).view(o.shape[0], -1))
        self.rot = stack.rotation(m.rotary)
        self.chunk_fits = not stack.f32 and ops.chunk_has_kernel(s.dim + s.rot, s.vdim)
        self.chunk_tc = self.chunk_fits and ops.chunk_tc_fits(s.dim, s.rot, s.vdim)

    def nbytes(self) -> int:
        return sum(x.nbytes() for x in (self.down, self.q_b, self.wo)) + (2 * self.k_b.numel() + self.v_b.numel()) * self.k_b.element_size()

    def workspace(self) -> dict[str, int]:
        return {"rows": self.down.n_out, "cq": self.sizes.q_rank, "q": self.q_b.n_out, "o": self.wo.k}

    def __call__(self, xn: torch.Tensor, fb, plan, kv, kv_layer: torch.Tensor) -> torch.Tensor:
        """Normed input rows -> the gated heads, input of the output product."""
        from ..ops import latent as ops
        st, m, s, T, lp = self.stack, self.m, self.sizes, xn.shape[0], plan.latent
        angles = plan.angles[self.rot]
        down = self.down(xn, st.ws("rows", T, self.down.n_out))
        gate = down[:, self.gate_col:] if m.gated else None
        cq = st.ws("cq", T, s.q_rank)
        ops.latent_prep(down, self.q_a_norm, self.kv_a_norm, angles, fb.positions, fb.seq_ids, fb.block_table, cq, kv_layer, m.rot_dim, s.latent, st.cfg.rms_eps)
        q = self.q_b(cq, st.ws("q", T, self.q_b.n_out)).view(T, s.heads, s.dim + s.rot)
        o = st.ws("o", T, self.wo.k)
        if lp.n_rows:
            self._attend_rows(q, o.view(T, s.heads, s.vdim), gate, angles, fb, lp, kv_layer)
        if lp.long:
            self._attend_chunks(q, o, gate, angles, fb, lp, kv_layer)
        return o

    def _attend_rows(self, q, o3, gate, angles, fb, lp: LatentPlan, kv_layer) -> None:
        n = lp.n_rows
        step = PLAIN_ROWS if lp.rows is None and n > PLAIN_ROWS else n
        for r0 in range(0, n, step):
            r1 = min(n, r0 + step)
            if lp.rows is not None:
                at = lp.rows.long()
                o3[at] = self._rows_values(q, q.index_select(0, at), lp.rows, None if gate is None else gate.index_select(0, at), angles, fb, lp, kv_layer,
                                           torch.empty(n, *o3.shape[1:], dtype=self.dtype, device=self.device))
            else:
                rows = torch.arange(r0, r1, dtype=torch.int32, device=self.device) if step < n else None
                self._rows_values(q, q[r0:r1], rows, None if gate is None else gate[r0:r1], angles, fb, lp, kv_layer, o3[r0:r1])

    def _rows_values(self, q, qs, rows, gate, angles, fb, lp: LatentPlan, kv_layer, out):
        """Attention values of single rows, gated, into ``out`` [rows, heads, vdim].  ``qs``: their queries; ``rows``: their tokens."""
        from ..ops import latent as ops
        st, m, s, n = self.stack, self.m, self.sizes, qs.shape[0]
        q_nope = qs[:, :, :s.dim].transpose(0, 1)
        q_lat, o_lat = (torch.empty(s.heads, n, s.latent, dtype=self.dtype, device=self.device) for _ in range(2))
        if ops.gemv_fits(self.k_bt, q_nope):
            ops.gemv_dense(self.k_bt, q_nope, q_lat)
        else:
            torch.bmm(q_nope, self.k_b, out=q_lat)
        max_keys = min(lp.max_keys, m.window) if m.window else lp.max_keys
        group = ops.rows_group(kv_layer, s.latent, m.rot_dim, s.heads, st.rows_tc)
        splits = ops.rows_splits(n, s.heads, group, st.rows_tc, max_keys, s.latent, st.part_o.numel())
        ops.latent_rows(q_lat, q, s.dim, angles, rows, fb.positions, fb.seq_ids, fb.block_table, kv_layer, m.rot_dim, m.window, m.scale, self.sink, o_lat,
                        st.part_o, st.part_ml, splits, group, st.status)
        side = (gate, 0, s.heads * s.vdim, None) if gate is not None else None
        if ops.gemv_fits(self.v_b, o_lat):
            ops.gemv_dense(self.v_b, o_lat, out.transpose(0, 1), act=ops.ACT_NONE if gate is None else ops.ACT_GATE, side=side)
        else:
            torch.bmm(o_lat, self.v_b.transpose(1, 2), out=out.transpose(0, 1))
            if gate is not None:
                flat = out.view(n, -1)
                ops.activate(flat, flat, ops.ACT_GATE, side)
        return out

    def _chunk_keys(self, lp: LatentPlan, window: int):
        """Sequence table of the prompt chunks for a window: which keys each needs and where they land in the key buffer."""
        got = lp.keys.get(window)
        if got is None:
            table, off, longest, max_q = [], 0, 0, 0
            for b, q0, n, ctx in lp.long:
                k0 = max(0, ctx - window + 1) if window else 0
                kn = ctx + n - k0
                table.append((b, q0, n, ctx, off, k0, kn, 0))
                off, longest, max_q = off + pad8(kn), max(longest, kn), max(max_q, n)
            got = lp.keys[window] = (torch.tensor(table, dtype=torch.int32, device=self.device), off, longest, max_q)
        return got

    def _attend_chunks(self, q, o, gate, angles, fb, lp: LatentPlan, kv_layer) -> None:
        from ..ops import latent as ops
        st, m, s = self.stack, self.m, self.sizes
        seqs, n_keys, longest, max_q = self._chunk_keys(lp, m.window)      # n_keys: with the rows up to the next multiple of 8
        lat = torch.empty(n_keys, s.width, dtype=self.dtype, device=self.device)
        ops.latent_gather(kv_layer, seqs, pad8(longest), fb.block_table, lat)
        c = lat[:, :s.latent]
        k = torch.mm(c, self.k_b.view(-1, s.latent).t())
        v_b = self.v_b.view(-1, s.latent)
        tc = self.chunk_tc and st.chunk_tc
        v = torch.mm(v_b, c.t()) if tc else torch.mm(c, v_b.t())
        ops.latent_chunk(q, angles, k, v, lat, s.latent, seqs, max_q, o, s.dim, s.rot, s.vdim, m.window, m.scale, self.sink, st.status if tc else None, gate)
