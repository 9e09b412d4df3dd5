"""Kernels of the recurrent mixers, of windowed attention and of the residual stream, each against plain double-precision forms."""
import pytest
import torch

from . import zogepel_oracle as oracle

pytestmark = pytest.mark.gpu
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64
EPS = 1e-5


def rnd(*shape, seed=0, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to("cuda")


def ints(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def err(got, want):
    want = want.double().cpu()
    return ((got.double().cpu() - want).abs().max() / want.abs().max().clamp_min(1e-30)).item()


# -- recurrences ---------------------------------------------------------------------------------------------------------------
class Recurrence:
    """Random rows for sequences of the given lengths and what both kernels take."""

    def __init__(self, lstm, heads, dim, vdim, lens, dtype, rot=0, decay=None, gate_shift=0.0, seed=0):
        self.lstm, self.H, self.d, self.v, self.lens, self.dtype = lstm, heads, dim, vdim, lens, dtype
        T, n = sum(lens), heads * dim
        self.rows = rnd(T, 2 * n + 2 * heads * vdim + 8, seed=seed).to(dtype)[:, :2 * n + 2 * heads * vdim]      # a row stride of its own
        self.offs = [0, n, 2 * n, 2 * n + heads * vdim]
        self.gates = (rnd(T, 2 * heads, seed=seed + 1, scale=2.0), rnd(heads, seed=seed + 2) + gate_shift, rnd(heads, seed=seed + 3) + 3.0 - gate_shift, 9.0) if lstm else None
        self.decay = None if lstm else torch.tensor(decay or [1 - 2.0 ** (-4 - 2 * h) for h in range(heads)], device="cuda")
        self.rot, self.norm = rot, 1 + rnd(heads * vdim, seed=seed + 4, scale=0.2) if lstm else None
        self.scale = dim ** -0.5
        slots = len(lens) + 2
        junk = lambda *s: torch.full(s, 7.0, device="cuda")                   # what a former owner left
        self.state = (junk(slots, heads, vdim, dim), junk(slots, heads, dim), junk(slots, heads)) if lstm else (junk(slots, heads, vdim, dim),)
        self.slots = torch.randperm(slots, generator=torch.Generator().manual_seed(seed))[:len(lens)].tolist()

    def run(self, lo, hi, chunked):
        """Rows lo[b] .. hi[b] of every sequence b as one batch; returns the normed and gated outputs per sequence."""
        from llaminar_b200.ops import dense, mixers
        from llaminar_b200 import ops
        at, pick, pos, cu = 0, [], [], [0]
        for b, n in enumerate(self.lens):
            pick += range(at + lo[b], at + hi[b])
            pos += range(lo[b], hi[b])
            cu.append(cu[-1] + hi[b] - lo[b])
            at += n
        rows = torch.empty(len(pick), self.rows.stride(0), dtype=self.dtype, device="cuda")[:, :self.rows.shape[1]]
        rows.copy_(self.rows[pick])
        gates = (self.gates[0][pick].contiguous(), *self.gates[1:]) if self.lstm else None
        angles = None
        if self.rot:
            f = torch.tensor([100.0 ** (-2 * i / self.rot) for i in range(self.rot // 2)], dtype=F64, device="cuda")
            angles = torch.empty(len(pick), self.rot // 2, 2, device="cuda")
            dense.rope_angles(ints(pos), f, 1.0, angles)
        out = torch.empty(len(pick), self.H * self.v, dtype=F32 if self.dtype == F32 else BF, device="cuda")
        args = (rows, self.offs, gates, self.decay, angles, self.scale if self.lstm else 1.0, 1.0 if self.lstm else self.scale, ints(cu), ints(pos), ints(self.slots),
                self.state, self.v, self.norm, not self.lstm, out, EPS)
        if chunked:
            status = ops.scratch_for(torch.device("cuda", 0)).status
            mixers.linear_chunk(*args, mixers.chunk_tables(cu, "cuda"), torch.empty_like(out), status)
            assert int(status[0]) == 0
        else:
            mixers.linear_rows(*args)
        return [out[cu[b]:cu[b + 1]] for b in range(len(self.lens))]

    def expected(self):
        """(outputs, final state) of every sequence."""
        res, at = [], 0
        for n in self.lens:
            x = self.rows[at:at + n].double().cpu()
            q, k, v, g = (x[:, a:a + self.H * w].reshape(n, self.H, w) for a, w in zip(self.offs, (self.d, self.d, self.v, self.v)))
            if self.lstm:
                z, bi, bf, cap = (t.double().cpu() if torch.is_tensor(t) else t for t in self.gates)
                z = z[at:at + n]
                eye = torch.eye(2 * self.H, dtype=F64)
                i, f = oracle.mlstm_gates(z, eye[:self.H], bi, eye[self.H:], bf, cap)
                o = oracle.mlstm_scan(q * self.scale, k, v, i, f)
                S, nn, m = torch.zeros(self.H, self.v, self.d, dtype=F64), torch.zeros(self.H, self.d, dtype=F64), torch.zeros(self.H, dtype=F64)
                for t in range(n):
                    top = torch.maximum(f[t] + m, i[t])
                    a, b = (f[t] + m - top).exp(), (i[t] - top).exp()
                    S, nn, m = a[:, None, None] * S + b[:, None, None] * v[t][:, :, None] * k[t][:, None], a[:, None] * nn + b[:, None] * k[t], top
                state = (S, nn, m)
                y = oracle.rms_divide(o, EPS).reshape(n, -1) * self.norm.double().cpu() * torch.sigmoid(g.reshape(n, -1))
            else:
                if self.rot:
                    q, k = (oracle.rotate(t, range(n), self.rot, 100.0) for t in (q, k))
                k, d = k * self.scale, self.decay.double().cpu()
                o = oracle.retention_scan(q, k, v, d)
                S = torch.zeros(self.H, self.v, self.d, dtype=F64)
                for t in range(n):
                    S = d[:, None, None] * S + v[t][:, :, None] * k[t][:, None]
                state = (S,)
                y = oracle.rms_divide(o, EPS).reshape(n, -1) * oracle.silu(g.reshape(n, -1))
            res.append((y, state))
            at += n
        return res

    def check(self, cuts, chunked, tol=None):
        """Feeds every sequence in the given fractions of its length and compares outputs and final state."""
        tol, state_tol = (tol or 2e-2, 1e-4) if self.dtype == BF else (1e-4, 1e-5)
        got = [[] for _ in self.lens]
        for a, b in zip(cuts, cuts[1:]):
            lo, hi = [int(a * n) for n in self.lens], [int(b * n) for n in self.lens]
            for i, o in enumerate(self.run(lo, hi, chunked)):
                got[i].append(o)
        for i, (y, state) in enumerate(self.expected()):
            o = torch.cat(got[i])
            assert torch.isfinite(o).all() and err(o, y) < tol, (i, err(o, y))
            for t, want in zip(self.state, state):
                assert err(t[self.slots[i]], want) < state_tol, (i, tuple(want.shape), err(t[self.slots[i]], want))


SIZES = [(2, 128, 256), (3, 48, 64), (1, 8, 8), (2, 64, 136), (2, 40, 272), (4, 16, 128)]


@pytest.mark.parametrize("heads,dim,vdim", SIZES)
@pytest.mark.parametrize("lens", [(300,), (5, 128, 129, 1, 260)])
def test_mlstm_over_prompts(heads, dim, vdim, lens):
    """State to 32-bit accuracy from bf16 rows; portions that end inside, at and behind a chunk."""
    for cuts in ([0, 1], [0, 0.43, 1]):
        if 1 in lens and len(cuts) > 2:
            continue
        Recurrence(True, heads, dim, vdim, lens, BF).check(cuts, True)


@pytest.mark.parametrize("heads,dim,vdim", SIZES)
@pytest.mark.parametrize("rot", [0.0, 0.5, 1.0])
def test_retention_over_prompts(heads, dim, vdim, rot):
    """Rotation of no, some and all values of a head, in whole 16-byte units and not."""
    r = int(dim * rot) // 2 * 2
    Recurrence(False, heads, dim, vdim, (5, 128, 129, 260), BF, rot=r).check([0, 1], True)
    Recurrence(False, heads, dim, vdim, (300,), BF, rot=max(2, r - 2) if r else 0).check([0, 0.43, 1], True)


def test_decays_at_their_limits():
    """(With nothing but its own key in the state, a row whose query is nearly orthogonal to it is all rounding of q and k: a wide
    tolerance on the bf16 outputs, none on the state.)"""
    Recurrence(False, 5, 32, 64, (200, 7), BF, rot=16, decay=[1.0, 0.0, 0.5, 0.01, 0.9999]).check([0, 0.6, 1], True, tol=0.3)
    Recurrence(False, 5, 32, 64, (200, 7), F32, rot=16, decay=[1.0, 0.0, 0.5, 0.01, 0.9999]).check([0, 0.6, 1], False)


@pytest.mark.parametrize("shift", [-14.0, 0.0, 14.0])
@pytest.mark.parametrize("chunked", [True, False])
def test_gates_at_their_limits(shift, chunked):
    """Input gates at their cap with forget gates shut, and the other way round."""
    Recurrence(True, 3, 64, 72, (200, 9), BF if chunked else F32, gate_shift=shift).check([0, 0.6, 1], chunked)


@pytest.mark.parametrize("lstm", [True, False])
@pytest.mark.parametrize("heads,dim,vdim", [*SIZES, (2, 200, 24), (1, 264, 1040)])
def test_rows_one_after_the_other(lstm, heads, dim, vdim):
    """32-bit rows; state rows spread over clusters of one to eight CTAs."""
    Recurrence(lstm, heads, dim, vdim, (3, 40, 1, 17), F32, rot=0 if lstm else 8).check([0, 1], False)


def test_rows_of_many_sequences():
    """A decode step's shape: so many sequences that a head is not spread."""
    r = Recurrence(True, 4, 32, 64, (2,) * 100, F32)
    r.check([0, 0.5, 1], False)


# -- attention -----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("heads,kv,dim,true_dim", [(4, 2, 64, 48), (6, 1, 128, 128), (3, 3, 128, 100), (4, 2, 40, 36)])
@pytest.mark.parametrize("window", [0, 1, 64, 65, 127, 300])
def test_attention_forms(heads, kv, dim, true_dim, window):
    """Prompt (tcgen05 and mma.sync), decode and plain kernel on pages in random order, behind cached context."""
    from llaminar_b200 import ops as base
    from llaminar_b200.ops import grouped as ops
    n, sc = 330, base.scratch_for(torch.device("cuda", 0))
    cols = (2 * heads + kv) * dim
    live = (torch.arange(cols, device="cuda") % dim) < true_dim                  # padding of a head is zero
    rows = (rnd(n, cols, seed=window) * live).to(BF)
    qn, kn, sink = 1.5 + rnd(heads * dim, seed=1, scale=0.2), 1.5 + rnd(kv * dim, seed=2, scale=0.2), rnd(heads, seed=3)
    pages = (n + 63) // 64
    bt = (torch.randperm(pages, generator=torch.Generator().manual_seed(1)).to(torch.int32) + 1).view(1, -1).cuda()
    cache, q = torch.zeros(pages + 1, 2, kv, 64, dim, dtype=BF, device="cuda"), torch.empty(n, heads, dim, dtype=BF, device="cuda")
    pos, sid = ints(list(range(n))), ints([0] * n)
    ops.attn_prep(rows, 0, heads * dim, heads * dim, qn, kn, pos, sid, bt, q, cache, true_dim, EPS)
    x = rows.double().cpu()
    cut = lambda t, h: t.reshape(n, h, dim)
    xq, xk = x[:, :heads * dim], x[:, heads * dim:(heads + kv) * dim]
    norm = lambda t, w, h: t / torch.sqrt((t * t).sum(-1, keepdim=True) / (h * true_dim) + EPS) * w.double().cpu()
    oq, ok = cut(norm(xq, qn, heads), heads), cut(norm(xk, kn, kv), kv)
    assert err(q, oq) < 1e-2 and err(cache[bt[0].long(), 0].permute(0, 2, 1, 3).reshape(-1, kv, dim)[:n], ok) < 1e-2
    assert torch.equal(cache[bt[0].long(), 1].permute(0, 2, 1, 3).reshape(-1, kv, dim)[:n], rows[:, heads * dim:(heads + kv) * dim].reshape(n, kv, dim))
    of, scale = [h // (heads // kv) for h in range(heads)], 0.7 / true_dim ** 0.5
    s = torch.einsum("thd,shd->hts", q.double().cpu(), cut(xk, kv)[:, of] * 0 + ok[:, of]) * scale
    s = s.masked_fill(~oracle.window_mask(n, window or 10 ** 6)[None], float("-inf"))
    o = torch.einsum("hts,shd->thd", oracle.softmax_with_sink(s, sink.double().cpu()), cut(xk, kv)[:, of]).reshape(n, -1)
    want = o * torch.sigmoid(x[:, (heads + kv) * dim:])
    gate = rows[:, (heads + kv) * dim:]
    out = torch.empty(n, heads * dim, dtype=BF, device="cuda")
    ops.attn_plain(q, cache, out, pos, sid, bt, window, scale, sink, gate)
    assert err(out, want) < 1e-2, "plain"
    if dim in ops.HEAD_SIZES:
        for first in (0, 70):                                                    # rows from `first` on, the ones before are context
            for status in ((sc.status, None) if dim == 128 else (None,)):
                part = torch.full((n - first, heads * dim), float("nan"), dtype=BF, device="cuda")
                g = gate[first:].clone() if first else gate
                ops.attn_prefill(q[first:].contiguous(), cache, part, bt, ints([0, n - first]), ints([first]), scale, n - first, window, sink, g, status)
                assert err(part, want[first:]) < 2e-2, ("prompt", first, status is not None)
        for last in (0, 63, 64, 65, 128, n - 1):
            for splits in (1, 3):
                one = torch.full((1, heads * dim), float("nan"), dtype=BF, device="cuda")
                ops.attn_decode(q[last:last + 1].contiguous(), cache, one, bt, ints([last + 1]), scale, splits, window, sink, gate[last:last + 1].float(), sc)
                assert err(one, want[last:last + 1]) < 2e-2, ("decode", last, splits)
        assert int(sc.status[0]) == 0


# -- residual stream -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("d", [33, 72, 1024, 1028, 4096, 5000, 8192, 9216])
def test_residual_updates(d, dtype):
    """Layer norm and RMSNorm behind a sublayer, both sides of a layer, the scaled embedding, the norm in front of the head."""
    from llaminar_b200.ops import dense as ops
    T, tol = 5, 1e-2 if dtype == BF else 1e-5
    y, y2, h0 = (rnd(T, d, seed=i).to(t) for i, t in ((1, dtype), (2, dtype), (3, F32)))
    y = y + 3                                                                    # a mean that has to be taken off
    w, wa, wb = (1 + rnd(d, seed=i, scale=0.3) for i in (4, 5, 6))
    D = lambda t: t.double().cpu()
    copy, xn = (torch.empty(T, d, dtype=dtype, device="cuda") for _ in range(2))
    for center in (True, False):
        f = oracle.layer_norm if center else oracle.rms_norm
        h = h0.clone()
        ops.resid_norm(h, y, w, copy0=copy, center_post=center, eps=EPS)
        want = D(h0) + f(D(y), D(w), EPS)
        assert err(h, want) < 1e-5 and err(copy, want) < tol
        h = h0.clone()
        ops.resid_norm(h, y, w, y2=y2, w_y=wa, w_y2=wb, copy0=copy, center_post=center, eps=EPS)
        want = D(h0) + f(0.5 * (oracle.rms_norm(D(y), D(wa), EPS) + oracle.rms_norm(D(y2), D(wb), EPS)), D(w), EPS)
        assert err(h, want) < 1e-5 and err(copy, want) < tol
        ops.resid_norm(h, w_next=w, xn=xn, center_next=center, eps=EPS)
        assert err(xn, f(D(h), D(w), EPS)) < tol
    table, tok = rnd(11, d, seed=7).to(dtype), ints([3, 0, 10, 3, 7])
    ops.resid_norm(h, table, None, add=False, y_rows=tok, factor=2.5, copy0=copy, eps=EPS)
    assert err(h, 2.5 * D(table)[tok.cpu().long()]) < 1e-6 and err(copy, 2.5 * D(table)[tok.cpu().long()]) < tol


@pytest.mark.parametrize("rows", [1, 3, 8, 16, 24, 33, 64])
def test_products_with_activations(rows):
    """Squared relu and the token's side input behind a product: fused (up to eight rows, or small matrices in groups of eight) and not."""
    from llaminar_b200.engine.dense import DenseLinear
    from llaminar_b200.ops import dense as ops
    for n, k in ((40, 64), (24, 56), (264, 320)):
        lin, x = DenseLinear(rnd(n, k, seed=n, scale=k ** -0.5).to(BF)), rnd(rows, k, seed=rows).to(BF)
        z = x.double().cpu() @ lin.w.double().cpu().T
        act, raw = torch.empty(rows, n, dtype=BF, device="cuda"), torch.empty(rows, n, dtype=BF, device="cuda")
        assert err(lin(x, raw), z) < 1e-2
        assert err(lin(x, torch.empty(rows, n, device="cuda")), z) < 1e-5
        assert err(lin.activated(x, act, raw, ops.ACT_RELU2), oracle.squared_relu(z)) < 2e-2
        table, tok = rnd(13, 3 * n, seed=5).to(BF), torch.randint(0, 13, (rows,), dtype=torch.int32).cuda()
        cols = n - 3                                                             # columns behind the side input's width give zero
        lin.activated(x, act, raw, ops.ACT_GELU_SIDE, (table, n + 1, cols, tok))
        e = table.double().cpu()[tok.cpu().long(), n + 1:n + 1 + cols]
        assert err(act[:, :cols], oracle.gelu_tanh(z[:, :cols]) * e) < 2e-2 and not act[:, cols:].any()
