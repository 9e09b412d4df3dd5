"""Kernels of latent-attention models against plain fp32 PyTorch: row and chunk attention in every form, norms, products."""
import math

import pytest
import torch

pytestmark = pytest.mark.gpu
BF = torch.bfloat16


def _rand(*shape, dtype=BF, scale=1.0, seed=0):
    g = torch.Generator(device="cuda").manual_seed(seed + sum(shape))
    return (torch.randn(*shape, device="cuda", generator=g) * scale).to(dtype)


def _turn(x, ang):
    """x [..., n] in fp32, ang [T, half, 2] broadcast over heads: pair (i, i + half)."""
    half = ang.shape[1]
    c, s = ang[..., 0], ang[..., 1]
    if x.dim() == 3:
        c, s = c[:, None], s[:, None]
    a, b = x[..., :half], x[..., half:2 * half]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., 2 * half:]], dim=-1)


class Cache:
    """A paged cache with random contents; page ids are shuffled over the pool."""

    def __init__(self, lens, latent, rot, width, dtype=BF, seed=0):
        P = max(-(-n // 64) for n in lens)
        n_pages = 3 + P * len(lens)
        perm = torch.randperm(n_pages - 1, generator=torch.Generator().manual_seed(seed)) + 1
        self.table = perm[:P * len(lens)].to(torch.int32).view(len(lens), P).contiguous().cuda()
        self.kv = _rand(n_pages, 64, width, dtype=dtype, seed=seed)
        self.kv[..., latent + rot:] = 0
        self.lens = lens

    def rows(self, s):
        n = self.lens[s]
        return self.kv[self.table[s].long()].reshape(-1, self.kv.shape[-1])[:n].float()


def _attend(q_lat, q_rot, kv, latent, rot, pos, window, scale, sink):
    """q_lat [H, L], q_rot [H, E] (rotated), kv [n, width] -> [H, L]"""
    lo = max(0, pos - window + 1) if window else 0
    k = kv[lo:pos + 1]
    s = (q_lat @ k[:, :latent].T + q_rot @ k[:, latent:latent + rot].T) * scale
    if sink is not None:
        s = torch.cat([s, sink[:, None]], -1)
    return torch.softmax(s, -1)[:, :k.shape[0]] @ k[:, :latent]


ROW_SIZES = [  # heads, latent, rot, half
    (5, 40, 8, 4), (16, 64, 32, 16), (7, 104, 24, 8), (20, 128, 16, 8), (16, 128, 64, 32), (32, 256, 32, 16), (40, 512, 64, 32), (12, 512, 64, 32)]


@pytest.mark.parametrize("heads,latent,rot,half", ROW_SIZES)
@pytest.mark.parametrize("form", ["auto", "mma", "plain", "f32"])
@pytest.mark.parametrize("window,sinks,splits", [(0, True, 1), (70, True, 3), (129, False, 2), (1, True, 1), (300, True, 7)])
def test_latent_rows(heads, latent, rot, half, form, window, sinks, splits):
    from llaminar_b200.ops import latent as ops
    dtype = torch.float32 if form == "f32" else BF
    width = (latent + rot + 15) // 16 * 16
    lens = [1, 64, 65, 127, 128, 129, 400, 513]
    c = Cache(lens, latent, rot, width, dtype, seed=heads)
    n, dim = len(lens), 24
    q = _rand(n, heads, dim + rot, dtype=dtype, seed=1)
    q_lat = _rand(heads, n, latent, dtype=dtype, seed=2, scale=2.0)
    pos = torch.tensor([x - 1 for x in lens], dtype=torch.int32, device="cuda")
    ang = _rand(n, half, 2, dtype=torch.float32, seed=3)
    sink = _rand(heads, dtype=torch.float32, seed=4) if sinks else None
    sid = torch.arange(n, dtype=torch.int32, device="cuda")
    group = 0 if form == "plain" else ops.rows_group(c.kv, latent, rot, heads, form == "auto")
    if form == "mma" and group == 0:
        pytest.skip("no mma.sync form for these sizes")
    out = torch.full_like(q_lat, float("nan"))
    po, pm = torch.full((1 << 23,), float("nan"), device="cuda"), torch.full((1 << 20,), float("nan"), device="cuda")
    status = torch.zeros(4, dtype=torch.int32, device="cuda")
    scale = 1 / math.sqrt(latent)
    ops.latent_rows(q_lat, q, dim, ang, None, pos, sid, c.table, c.kv, rot, window, scale, sink, out, po, pm, splits if group else 1, group, status)
    torch.cuda.synchronize()
    assert int(status[0]) == 0
    qr = _turn(q[..., dim:].float(), ang)
    tol = 2e-5 if form == "f32" else 2e-2
    for i in range(n):
        ref = _attend(q_lat[:, i].float(), qr[i], c.rows(i), latent, rot, lens[i] - 1, window, scale, sink)
        err = (out[:, i].float() - ref).abs().max().item()
        assert err < tol * max(1.0, ref.abs().max().item()), (i, err)


@pytest.mark.parametrize("tensor_core", [False, True])
@pytest.mark.parametrize("heads,dim,rot,vdim,half", [(3, 24, 8, 16, 4), (2, 64, 64, 64, 32), (4, 128, 64, 128, 32), (3, 48, 16, 80, 8), (2, 96, 32, 112, 16), (2, 160, 48, 136, 8)])
@pytest.mark.parametrize("window,sinks", [(0, True), (50, True), (128, False), (300, True), (1, True)])
def test_latent_chunk(tensor_core, heads, dim, rot, vdim, half, window, sinks):
    from llaminar_b200.ops import latent as ops
    if tensor_core and not ops.chunk_tc_fits(dim, rot, vdim):
        pytest.skip("no tcgen05 form for these sizes")
    latent = 40
    width = (latent + rot + 15) // 16 * 16
    seqs = [(0, 9), (0, 400), (63, 130), (700, 257), (5, 64)]                 # (context, rows)
    table, off, q0, T = [], 0, 0, sum(n for _, n in seqs)
    for b, (ctx, n) in enumerate(seqs):
        k0 = max(0, ctx - window + 1) if window else 0
        table.append((b, q0, n, ctx, off, k0, ctx + n - k0, 0))
        off, q0 = off + (ctx + n - k0 + 7) // 8 * 8, q0 + n
    k, v, lat = _rand(off, heads * dim, seed=1), _rand(off, heads * vdim, seed=2), _rand(off, width, seed=3)
    q, ang = _rand(T, heads, dim + rot, seed=4), _rand(T, half, 2, dtype=torch.float32, seed=5)
    sink = _rand(heads, dtype=torch.float32, seed=6) if sinks else None
    out = torch.full((T, heads * vdim), float("nan"), dtype=BF, device="cuda")
    status = torch.zeros(4, dtype=torch.int32, device="cuda")
    scale = (dim + rot) ** -0.5
    ops.latent_chunk(q, ang, k, v.t().contiguous() if tensor_core else v, lat, latent, torch.tensor(table, dtype=torch.int32, device="cuda"),
                     max(n for _, n in seqs), out, dim, rot, vdim, window, scale, sink, status if tensor_core else None)
    torch.cuda.synchronize()
    assert int(status[0]) == 0
    qf = torch.cat([q[..., :dim].float(), _turn(q[..., dim:].float(), ang).to(BF).float()], -1)
    o3 = out.view(T, heads, vdim).float()
    for b, q0, n, ctx, o, k0, kn, _ in table:
        kk = torch.cat([k[o:o + kn].view(kn, heads, dim), lat[o:o + kn, None, latent:latent + rot].expand(-1, heads, -1)], -1).float()
        s = torch.einsum("thd,shd->hts", qf[q0:q0 + n], kk) * scale
        i, j = torch.arange(ctx, ctx + n, device="cuda")[:, None], torch.arange(k0, k0 + kn, device="cuda")[None]
        seen = (j <= i) & ((i - j < window) if window else torch.ones_like(j <= i))
        s = s.masked_fill(~seen[None], float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink[:, None, None].expand(-1, n, 1)], -1)
        ref = torch.einsum("hts,shv->thv", torch.softmax(s, -1)[..., :kn], v[o:o + kn].view(kn, heads, vdim).float())
        err = (o3[q0:q0 + n] - ref).abs().max().item()
        assert err < 2.5e-2 * max(1.0, ref.abs().max().item()), (b, err)


@pytest.mark.parametrize("dtype", [BF, torch.float32])
@pytest.mark.parametrize("q_rank,kv_rank,rot,half", [(72, 104, 24, 8), (33, 50, 12, 4), (1536, 512, 64, 32), (24, 40, 8, 2)])
def test_latent_prep_and_gather(dtype, q_rank, kv_rank, rot, half):
    from llaminar_b200.ops import latent as ops
    T, off = 150, -(-kv_rank // 8) * 8
    width, qp = (off + -(-rot // 8) * 8 + 15) // 16 * 16, -(-q_rank // 8) * 8
    lens = [100, 50]
    c = Cache(lens, off, width - off, width, dtype)
    down = _rand(T, q_rank + kv_rank + rot, dtype=dtype, seed=1)
    qn, kn = _rand(q_rank, dtype=torch.float32, seed=2), _rand(kv_rank, dtype=torch.float32, seed=3)
    ang = _rand(T, half, 2, dtype=torch.float32, seed=4)
    pos = torch.cat([torch.arange(100), torch.arange(50)]).to(torch.int32).cuda()
    sid = torch.cat([torch.zeros(100), torch.ones(50)]).to(torch.int32).cuda()
    cq = torch.full((T, qp), float("nan"), dtype=dtype, device="cuda")
    ops.latent_prep(down, qn, kn, ang, pos, sid, c.table, cq, c.kv, rot, off, 1e-5)
    f = down.float()
    norm = lambda x, w: x / torch.sqrt((x * x).mean(-1, keepdim=True) + 1e-5) * w
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == BF else dict(rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(cq[:, :q_rank].float(), norm(f[:, :q_rank], qn), **tol)
    assert not cq[:, q_rank:].any()
    want = torch.zeros(T, width, device="cuda")
    want[:, :kv_rank] = norm(f[:, q_rank:q_rank + kv_rank], kn)
    want[:, off:off + rot] = _turn(f[:, q_rank + kv_rank:], ang)
    got = torch.cat([c.rows(0), c.rows(1)])
    torch.testing.assert_close(got, want, **tol)
    seqs = torch.tensor([[0, 0, 60, 40, 0, 13, 87, 0], [1, 60, 20, 30, 88, 0, 50, 0]], dtype=torch.int32, device="cuda")
    out = torch.full((88 + 56, width), float("nan"), dtype=dtype, device="cuda")
    ops.latent_gather(c.kv, seqs, 88, c.table, out)
    assert torch.equal(out[:87].float(), c.rows(0)[13:]) and torch.equal(out[88:138].float(), c.rows(1))
    assert not out[87].any() and not out[138:].any()


@pytest.mark.parametrize("dtype", [BF, torch.float32])
@pytest.mark.parametrize("d", [33, 256, 4096, 5000])
def test_resid_norm(dtype, d):
    from llaminar_b200.ops import latent as ops
    T = 7
    h0, y = _rand(T, d, dtype=torch.float32, seed=1), _rand(20, d, dtype=dtype, seed=2)
    wp, wn = _rand(d, dtype=torch.float32, seed=3), _rand(d, dtype=torch.float32, seed=4)
    norm = lambda x, w: x / torch.sqrt((x * x).mean(-1, keepdim=True) + 1e-6) * w
    rows = torch.tensor([3, 19, 0, 3, 7, 8, 1], dtype=torch.int32, device="cuda")
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == BF else dict(rtol=1e-5, atol=1e-5)
    for add in (True, False):
        h, xn, cat = h0.clone(), torch.empty(T, d, dtype=dtype, device="cuda"), torch.zeros(T, 2 * d, dtype=dtype, device="cuda")
        ops.resid_norm(h, y, wp, add=add, y_rows=rows, w_next=wn, xn=xn, copy0=cat[:, d:], copy1=cat[:, :d], eps=1e-6)
        want = norm(y.float()[rows.long()], wp) + (h0 if add else 0)
        torch.testing.assert_close(h, want, rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(xn.float(), norm(want, wn), **tol)
        torch.testing.assert_close(cat.float(), torch.cat([want, want], 1), **tol)
    h, xn = h0.clone(), torch.empty(T, d, dtype=dtype, device="cuda")
    ops.resid_norm(h, w_next=wn, xn=xn, eps=1e-6)
    assert torch.equal(h, h0)
    torch.testing.assert_close(xn.float(), norm(h0, wn), **tol)


@pytest.mark.parametrize("m", [1, 3, 4, 8])
@pytest.mark.parametrize("z,n,k", [(1, 300, 64), (1, 1000, 4096), (5, 96, 128), (3, 64, 40), (1, 7, 200)])
def test_gemv_dense(m, z, n, k):
    from llaminar_b200.ops import latent as ops
    w, x = _rand(z, n, k, seed=1, scale=k ** -0.5), _rand(z, m, k, seed=2)
    ref = torch.einsum("znk,zmk->zmn", w.float(), x.float())
    for dt in (BF, torch.float32):
        out = torch.empty(z, m, n, dtype=dt, device="cuda")
        ops.gemv_dense(w, x, out)
        torch.testing.assert_close(out.float(), ref, rtol=1e-2, atol=1e-2 if dt == BF else 1e-4)
    if n % 2 == 0:
        act = torch.empty(z, m, n // 2, dtype=BF, device="cuda")
        ops.gemv_dense(w, x, act, gelu=True)
        want = torch.nn.functional.gelu(ref[..., :n // 2], approximate="tanh") * ref[..., n // 2:]
        torch.testing.assert_close(act.float(), want, rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("dtype", [BF, torch.float32])
@pytest.mark.parametrize("ff", [56, 33, 1024])
def test_gelu_mul(dtype, ff):
    from llaminar_b200.ops import latent as ops
    gu = _rand(9, 2 * ff, dtype=dtype, seed=1, scale=2.0)
    act = torch.empty(9, ff, dtype=dtype, device="cuda")
    ops.gelu_mul(gu, act)
    f = gu.float()
    want = torch.nn.functional.gelu(f[:, :ff], approximate="tanh") * f[:, ff:]
    torch.testing.assert_close(act.float(), want, rtol=1e-2 if dtype == BF else 1e-5, atol=1e-2 if dtype == BF else 1e-5)


def test_rope_angles_far_positions():
    from llaminar_b200.models.config import Rotary
    from llaminar_b200.ops import latent as ops
    r = Rotary(16, 1e4)
    pos = torch.tensor([0, 1, 1000, 123457, 1048575], dtype=torch.int32, device="cuda")
    f = torch.tensor(r.frequencies(), dtype=torch.float64, device="cuda")
    out = torch.empty(5, 8, 2, device="cuda")
    ops.rope_angles(pos, f, 1.25, out)
    a = pos.double()[:, None] * f
    torch.testing.assert_close(out, (torch.stack([a.cos(), a.sin()], -1) * 1.25).float(), rtol=1e-6, atol=1e-6)
