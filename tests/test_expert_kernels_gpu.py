"""Kernels of routed experts and of grouped attention, each against plain double-precision forms."""
import pytest
import torch

from . import kefasun_oracle as oracle

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


def status():
    from llaminar_b200 import ops
    return ops.scratch_for(torch.device("cuda", 0)).status


# -- experts -------------------------------------------------------------------------------------------------------------------
class Layer:
    """Random experts, and the pairs' outputs in double precision from the kernel's own choice."""

    def __init__(self, T, E, top, d, ff, dtype=BF, seed=0, skew=0.0):
        self.T, self.E, self.top, self.d, self.ff, self.dtype = T, E, top, d, ff, dtype
        self.x, self.router = rnd(T, d, seed=seed).to(dtype), rnd(E, d, seed=seed + 1, scale=3 * d ** -0.5).to(dtype)
        self.gu, self.down = rnd(E, 2 * ff, d, seed=seed + 2, scale=d ** -0.5).to(dtype), rnd(E, d, ff, seed=seed + 3, scale=ff ** -0.5).to(dtype)
        self.bias = rnd(E, seed=seed + 4) + skew * torch.arange(E, device="cuda")
        self.ids = torch.full((T, top), -1, dtype=torch.int32, device="cuda")
        self.w = torch.full((T, top), float("nan"), device="cuda")
        self.act, self.y = (torch.full((T * top, n), float("nan"), dtype=dtype, device="cuda") for n in (ff, d))

    def check_choice(self):
        T = lambda name: {"router": self.router.double().cpu(), "router.b": self.bias.double().cpu()}[name]
        ids, w = oracle.route(self.x.double().cpu(), T, self.top)
        clear = oracle.router_gap(self.x.double().cpu(), T, self.top) > 1e-4
        assert clear.float().mean() > 0.9
        a, b = self.ids.cpu().long().sort(-1), ids.sort(-1)
        assert torch.equal(a.values[clear], b.values[clear])
        assert (self.w.double().cpu().gather(1, a.indices) - w.gather(1, b.indices))[clear].abs().max() < 1e-5

    def expected(self, picks):
        """Activations and outputs of the given pairs."""
        acts, ys = [], []
        for p in picks:
            e, x = int(self.ids.view(-1)[p]), self.x[p // self.top].double()
            h = self.gu[e].double() @ x
            acts.append(oracle.silu(h[:self.ff]) * h[self.ff:])
            ys.append(self.down[e].double() @ acts[-1])
        return torch.stack(acts), torch.stack(ys)

    def check(self, place=None, tol=1e-2):
        picks = list(range(0, self.T * self.top, max(1, self.T * self.top // 200)))
        rows = picks if place is None else place[picks].long()
        act, y = self.expected(picks)
        assert torch.isfinite(self.y).all() and err(self.act[rows], act) < tol and err(self.y[rows], y) < tol, (err(self.act[rows], act), err(self.y[rows], y))


# tokens, experts, chosen, width, expert width: one expert, all chosen, odd numbers of experts, tails of the MMA steps and tiles, more than
# one tile per expert, experts without tokens
SIZES = [(1, 8, 2, 256, 104), (5, 6, 3, 200, 72), (7, 40, 5, 136, 8), (33, 1, 1, 64, 64), (130, 5, 2, 1000, 200), (60, 3, 3, 128, 264), (300, 130, 2, 72, 136), (500, 4, 1, 512, 320), (9, 200, 6, 64, 16)]


@pytest.mark.parametrize("T,E,top,d,ff", SIZES)
def test_few_pairs(T, E, top, d, ff):
    from llaminar_b200.ops import experts as ops
    x = Layer(T, E, top, d, ff)
    ops.expert_route(x.bias, x.ids, x.w, x=x.x, router=x.router)
    x.check_choice()
    if T * top > ops.max_pairs():
        return
    ops.expert_rows(x.gu, x.x, x.ids, x.act, top, True)
    ops.expert_rows(x.down, x.act, x.ids, x.y, 1, False)
    x.check()


@pytest.mark.parametrize("T,E,top,d,ff", SIZES + [(1500, 8, 4, 256, 96), (900, 16, 1, 192, 520)])
@pytest.mark.parametrize("skew", [0.0, 1.5])
def test_sorted_pairs(T, E, top, d, ff, skew):
    """Tiles of 128 rows that end inside, at and behind an expert's last row; with a skew some experts get no token at all."""
    from llaminar_b200.ops import experts as ops
    x = Layer(T, E, top, d, ff, skew=skew)
    P = T * top
    counts, ranks, place = torch.zeros(E, dtype=torch.int32, device="cuda"), torch.full((P,), -1, dtype=torch.int32, device="cuda"), torch.full((P,), -1, dtype=torch.int32, device="cuda")
    xs = torch.full((P, d), float("nan"), dtype=BF, device="cuda")
    ops.expert_route(x.bias, x.ids, x.w, logits=torch.mm(x.x, x.router.t(), out_dtype=F32), counts=counts, ranks=ranks)
    x.check_choice()
    ops.expert_place(x.x, x.ids, ranks, counts, place, xs)
    assert torch.equal(counts.cpu(), torch.bincount(x.ids.view(-1).cpu(), minlength=E).int())
    assert torch.equal(place.sort().values.cpu(), torch.arange(P, dtype=torch.int32))                    # every row once, experts in order
    order = x.ids.view(-1)[place.argsort()]
    assert bool((order[1:] >= order[:-1]).all()) and torch.equal(xs[place.long()], x.x.repeat_interleave(top, 0))
    ops.expert_grouped(x.gu, xs, counts, x.act, True, status())
    ops.expert_grouped(x.down, x.act, counts, x.y, False, status())
    assert int(status()[0]) == 0
    x.check(place)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,E,top,d,ff", [(9, 6, 3, 33, 17), (70, 5, 2, 136, 24)])
def test_any_size_in_float_arithmetic(T, E, top, d, ff, dtype):
    from llaminar_b200.ops import experts as ops
    x = Layer(T, E, top, d, ff, dtype)
    ops.expert_route(x.bias, x.ids, x.w, x=x.x, router=x.router)
    x.check_choice()
    ops.expert_plain(x.gu, x.x, x.ids, x.act, top, True)
    ops.expert_plain(x.down, x.act, x.ids, x.y, 1, False)
    x.check(tol=1e-2 if dtype == BF else 1e-5)


def test_equal_logits_and_broken_logits_name_valid_experts():
    from llaminar_b200.ops import experts as ops
    ids, w = torch.empty(3, 4, dtype=torch.int32, device="cuda"), torch.empty(3, 4, device="cuda")
    z = torch.zeros(3, 9, device="cuda")
    z[1], z[2] = float("nan"), float("-inf")
    ops.expert_route(torch.zeros(9, device="cuda"), ids, w, logits=z)
    assert ids[0].tolist() == [0, 1, 2, 3] and torch.allclose(w[0], torch.full((4,), 0.25, device="cuda"))
    assert bool(((ids >= 0) & (ids < 9)).all())


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("d", [64, 1024, 4096, 8192, 9000, 33])
@pytest.mark.parametrize("sorted_rows", [True, False])
def test_residual_norm_sums_weighted_parts(d, dtype, sorted_rows):
    from llaminar_b200.ops import dense as ops
    T, n = 5, 3
    h, y, wt = rnd(T, d), rnd(T * n, d, seed=1).to(dtype), rnd(T, n, seed=2).abs()
    rows = torch.randperm(T * n, generator=torch.Generator().manual_seed(3)).int().cuda() if sorted_rows else None
    post, nxt, xn = 1 + rnd(d, seed=4, scale=0.1), 1 + rnd(d, seed=5, scale=0.1), torch.empty(T, d, dtype=dtype, device="cuda")
    v = (y.double() if rows is None else y.double()[rows.long()]).view(T, n, d)
    want = h.double() + oracle.rms_norm((v * wt.double()[..., None]).sum(1), post.double(), EPS)
    ops.resid_norm(h, y, post, w_next=nxt, xn=xn, eps=EPS, y_rows=rows, y_w=wt)
    assert err(h, want) < 1e-5 and err(xn, oracle.rms_norm(want, nxt.double(), EPS)) < (1e-2 if dtype == BF else 1e-5)


# -- activations and gates --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("n", [64, 1030, 33])
def test_silu_pairs_and_gates(n, dtype):
    from llaminar_b200.ops import dense as ops
    T, tol = 7, 1e-2 if dtype == BF else 1e-5
    x, act = rnd(T, 2 * n, seed=1, scale=3.0).to(dtype), torch.empty(T, n, dtype=dtype, device="cuda")
    ops.activate(x, act, ops.ACT_SILU_MUL)
    assert err(act, oracle.silu(x[:, :n].double()) * x[:, n:].double()) < tol
    wide = rnd(T, 3 * n + 5, seed=2).to(dtype)
    o, gate = act.clone(), wide[:, 5:5 + n]                         # in place, gate columns inside wider rows
    ops.activate(o, o, ops.ACT_GATE, (gate, 0, n, None))
    assert err(o, act.double() * torch.sigmoid(gate.double())) < tol


@pytest.mark.parametrize("m", [1, 3, 8])
def test_small_products_with_silu_and_gates(m):
    from llaminar_b200.ops import dense as ops
    k, ff, z, n = 200, 120, 3, 40
    x, w = rnd(m, k).to(BF), rnd(2 * ff, k, seed=1, scale=k ** -0.5).to(BF)
    out = torch.empty(m, ff, dtype=BF, device="cuda")
    ops.gemv_dense(w[None], x[None], out[None], act=ops.ACT_SILU_MUL)
    f = x.double() @ w.double().T
    assert err(out, oracle.silu(f[:, :ff]) * f[:, ff:]) < 2e-2
    x, w, gate = rnd(z, m, k, seed=2).to(BF), rnd(z, n, k, seed=3, scale=k ** -0.5).to(BF), rnd(m, z * n + 8, seed=4).to(BF)[:, 8:]
    out = torch.empty(m, z, n, dtype=BF, device="cuda")
    ops.gemv_dense(w, x, out.transpose(0, 1), act=ops.ACT_GATE, side=(gate, 0, z * n, None))
    want = torch.einsum("zmk,znk->mzn", x.double(), w.double()) * torch.sigmoid(gate.double()).view(m, z, n)
    assert err(out, want) < 2e-2


# -- grouped attention -------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,rows_dtype", [(BF, BF), (BF, F32), (F32, F32)])
@pytest.mark.parametrize("heads,kv,dim,true_dim,rot", [(4, 2, 64, 48, 20), (6, 1, 128, 128, 128), (3, 3, 128, 100, 2), (9, 3, 40, 36, 36), (2, 1, 200, 193, 64)])
def test_head_prep(heads, kv, dim, true_dim, rot, dtype, rows_dtype):
    from llaminar_b200.ops import dense, grouped as ops
    n = 150
    live = torch.arange(dim, device="cuda") < true_dim
    rows = (rnd(n, heads + 2 * kv, dim) * live).reshape(n, -1).to(rows_dtype)
    qn, kn = ((1.5 + rnd(dim, seed=s, scale=0.3)) * live for s in (1, 2))
    pages = (n + 63) // 64
    bt = (torch.randperm(pages, generator=torch.Generator().manual_seed(1)).to(torch.int32) + 1).view(1, -1).cuda()
    cache, q = torch.full((pages + 1, 2, kv, 64, dim), 7.0, dtype=dtype, device="cuda"), torch.empty(n, heads, dim, dtype=dtype, device="cuda")
    f = torch.tensor([100.0 ** (-2 * i / rot) for i in range(rot // 2)], dtype=F64, device="cuda")
    ang, pos = torch.empty(n, rot // 2, 2, device="cuda"), ints(list(range(n)))
    dense.rope_angles(pos, f, 1.0, ang)
    ops.head_prep(rows, 0, heads * dim, (heads + kv) * dim, qn, kn, ang, pos, ints([0] * n), bt, q, cache, true_dim, EPS)
    x = rows.double().cpu().view(n, heads + 2 * kv, dim)

    def want(v, gain):
        v = v / torch.sqrt((v * v).sum(-1, keepdim=True) / true_dim + EPS) * gain.double().cpu()
        return oracle.rotate_halves(v.transpose(0, 1), range(n), {"dims": rot, "base": 100.0}).transpose(0, 1)
    tol = 1e-2 if dtype == BF else 1e-5
    flat = lambda which: cache[bt[0].long(), which].permute(0, 2, 1, 3).reshape(-1, kv, dim)[:n]
    assert err(q, want(x[:, :heads], qn)) < tol and err(flat(0), want(x[:, heads:heads + kv], kn)) < tol
    assert torch.equal(flat(1), rows.view(n, -1, dim)[:, heads + kv:].to(dtype))
    assert bool((cache[0] == 7.0).all())                            # the scratch page, and the rows behind the last token
    assert bool((cache[bt[0, -1].long(), :, :, n % 64:] == 7.0).all())


@pytest.mark.parametrize("heads,kv,dim,true_dim", [(4, 2, 64, 48), (6, 1, 128, 128), (3, 3, 128, 100), (4, 2, 40, 36)])
@pytest.mark.parametrize("chunk,window,cap,gate_kind,sink_kind", [(1, 0, 0.0, "head", True), (64, 0, 0.0, "head", True), (65, 0, 9.0, "value", False), (127, 50, 0.0, "", True),
                                                                  (300, 0, 4.0, "head", False), (0, 0, 3.0, "value", False), (0, 70, 5.0, "", True)])
def test_attention_forms(heads, kv, dim, true_dim, chunk, window, cap, gate_kind, sink_kind):
    """Prompt (tcgen05 and mma.sync), decode and plain kernel on pages in random order, behind cached context."""
    from llaminar_b200 import ops as base
    from llaminar_b200.ops import grouped as ops
    n, sc = 330, base.scratch_for(torch.device("cuda", 0))
    live = torch.arange(dim, device="cuda") < true_dim
    q, k, v = ((rnd(n, h, dim, seed=chunk + s) * live).to(BF) for h, s in ((heads, 0), (kv, 1), (kv, 2)))
    pages = (n + 63) // 64
    bt = (torch.randperm(pages, generator=torch.Generator().manual_seed(1)).to(torch.int32) + 1).view(1, -1).cuda()
    cache = torch.zeros(pages + 1, 2, kv, 64, dim, dtype=BF, device="cuda")
    for i in range(n):
        cache[bt[0, i // 64].long(), 0, :, i % 64], cache[bt[0, i // 64].long(), 1, :, i % 64] = k[i], v[i]
    sink = torch.zeros(heads, device="cuda") if sink_kind else None
    cols = {"head": heads, "value": heads * dim, "": 0}[gate_kind]
    gate = rnd(n, cols + 16, seed=9, scale=2.0).to(BF)[:, 16:] if cols else None
    scale, of = 2.0 / true_dim ** 0.5, [h // (heads // kv) for h in range(heads)]
    x = lambda t: t.double().cpu()
    s = torch.einsum("thd,shd->hts", x(q), x(k)[:, of]) * scale
    s = oracle.soft_cap(s, cap) if cap else s
    seen = oracle.causal_mask(n)
    seen = seen & oracle.chunk_mask(n, chunk) if chunk else seen
    seen = seen & oracle.window_mask(n, window) if window else seen
    s = s.masked_fill(~seen[None], float("-inf"))
    p = oracle.softmax_plus_one(s) if sink_kind else torch.softmax(s, -1)
    want = torch.einsum("hts,shd->thd", p, x(v)[:, of])
    if gate_kind == "head":
        want = oracle.head_gate(want, x(gate))
    elif gate_kind:
        want = oracle.value_gate(want, x(gate))
    want, how = want.reshape(n, -1), dict(chunk=chunk, softcap=cap)
    pos, sid, out = ints(list(range(n))), ints([0] * n), torch.empty(n, heads * dim, dtype=BF, device="cuda")
    ops.attn_plain(q, cache, out, pos, sid, bt, window, scale, sink, gate, **how)
    assert err(out, want) < 1e-2, "plain"
    if dim not in ops.HEAD_SIZES:
        return
    for first in (0, 70, 128):                                      # rows from `first` on, the ones before are context
        for st in ((sc.status, None) if dim == 128 else (None,)):
            part = torch.full((n - first, heads * dim), float("nan"), dtype=BF, device="cuda")
            g = gate[first:] if gate is not None else None
            if gate_kind == "value" and first:
                g = torch.empty(n - first, cols + 16, dtype=BF, device="cuda")[:, 16:].copy_(g)
            ops.attn_prefill(q[first:].contiguous(), cache, part, bt, ints([0, n - first]), ints([first]), scale, n - first, window, sink, g, st, **how)
            assert err(part, want[first:]) < 2e-2, ("prompt", first, st is not None, err(part, want[first:]))
    for last in (0, 63, 64, 65, 128, n - 1):
        for splits in (1, 3):
            one = torch.full((1, heads * dim), float("nan"), dtype=BF, device="cuda")
            g = gate[last:last + 1].float() if gate is not None else None
            ops.attn_decode(q[last:last + 1].contiguous(), cache, one, bt, ints([last + 1]), scale, splits, window, sink, g, sc, **how)
            assert err(one, want[last:last + 1]) < 2e-2, ("decode", last, splits)
    assert int(sc.status[0]) == 0
