"""Kernels of parallel layers, each against plain double-precision forms: averages over depth, convolved projections, lightning attention,
grouped routing, limited experts."""
import pytest
import torch

from . import lagedra_oracle as oracle

pytestmark = pytest.mark.gpu
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64
EPS = 1e-5
both = pytest.mark.parametrize("dtype", [BF, F32])


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


# -- residual updates ----------------------------------------------------------------------------------------------------------
@both
@pytest.mark.parametrize("d", [64, 1020, 1024, 2048, 4096, 8192, 12000, 33])
@pytest.mark.parametrize("n_past", [0, 1, 5, 9])
def test_depth_mix(d, n_past, dtype):
    from llaminar_b200.ops import dense as ops
    T, parts, streams = 5, 3, n_past + 1
    tol = 1e-2 if dtype == BF else 1e-5
    for kind in ("rows", "parts", "last", "gather"):
        room = torch.full((streams if kind != "last" else n_past, T + 2, d), 7.0, device="cuda")        # streams of more rows than this call has
        past = room[:, :T]
        past[:n_past] = rnd(n_past, T, d, seed=1)
        h, w, y = rnd(T, d, seed=2), rnd(n_past + 1, seed=3), rnd(T + 4, d, seed=4).to(dtype)
        gains = [1 + rnd(1, seed=5), 1 + rnd(1, seed=6)] if kind != "last" else [rnd(d, seed=5)]
        outs = [torch.empty(T, d, dtype=dtype, device="cuda") for _ in gains]
        kw, x = {}, h.double()
        if kind == "gather":
            rows, pos, z = ints([3, 0, 8, 8, 1]), ints([0, 7, 2, 2, 5]), rnd(9, d, seed=7).to(dtype)
            kw, x = dict(add=False, y_rows=rows, z=z, z_rows=pos), y.double()[rows.long()] + z.double()[pos.long()]
        elif kind == "parts":
            z, rows, wt = rnd(T * parts, d, seed=7).to(dtype), torch.randperm(T * parts, generator=torch.Generator().manual_seed(8)).int().cuda(), rnd(T, parts, seed=9).abs()
            kw, x = dict(z=z, z_rows=rows, z_w=wt), x + y[:T].double() + (z.double()[rows.long()].view(T, parts, d) * wt.double()[..., None]).sum(1)
        else:
            z = rnd(T, d, seed=7).to(dtype)
            kw, x = dict(z=z), x + y[:T].double() + z.double()
        want = oracle.depth_average([*past[:n_past].double(), x], w.double())
        if kind == "last" and n_past == 0:
            continue
        ops.depth_mix(h, y if kind == "gather" else y[:T], **kw, past=past, n_past=n_past, w=w, norms=list(zip(gains, outs)), eps=EPS)
        assert err(h, want) < 1e-5 and (kind == "last" or err(past[n_past], x) < 1e-5) and bool((room[:, T:] == 7).all())
        for g, o in zip(gains, outs):
            assert err(o, oracle.scalar_norm(want, g.double(), EPS)) < tol


@both
def test_depth_mix_only_reads_or_has_no_streams(dtype):
    from llaminar_b200.ops import dense as ops
    h, y, g, xn = rnd(4, 96), rnd(4, 96, seed=1).to(dtype), rnd(1, seed=2), torch.empty(4, 96, dtype=dtype, device="cuda")
    keep = h.clone()
    ops.depth_mix(h, norms=[(g, xn)], eps=EPS)
    assert torch.equal(h, keep) and err(xn, oracle.scalar_norm(h.double(), g.double(), EPS)) < 1e-2
    ops.depth_mix(h, y, eps=EPS)
    assert err(h, keep.double() + y.double()) < 1e-6


@both
@pytest.mark.parametrize("n", [64, 1030, 33])
def test_ungated_activations_on_rows_of_a_wider_matrix(n, dtype):
    from llaminar_b200.ops import dense as ops
    x, out = rnd(7, n + 24).to(dtype), torch.empty(7, n, dtype=dtype, device="cuda")
    tail = x[:, n:].clone()
    for kind, f in ((ops.ACT_GELU, oracle.gelu_tanh), (ops.ACT_SILU, oracle.silu)):
        ops.activate(x[:, :n], out, kind)
        assert err(out, f(x[:, :n].double())) < (1e-2 if dtype == BF else 1e-5)
    want = oracle.silu(x[:, :n].double())
    ops.activate(x[:, :n], x[:, :n], ops.ACT_SILU)
    assert err(x[:, :n], want) < 1e-2 and torch.equal(x[:, n:], tail)


@pytest.mark.parametrize("rows", [1, 5, 8])
def test_gelu_behind_a_small_product(rows):
    from llaminar_b200.ops import dense as ops
    w, x, out = rnd(200, 136, scale=136 ** -0.5).bfloat16(), rnd(rows, 136, seed=1).bfloat16(), torch.empty(rows, 200, dtype=BF, device="cuda")
    ops.gemv_dense(w[None], x[None], out[None], act=ops.ACT_GELU)
    assert err(out, oracle.gelu_tanh(x.double() @ w.double().T)) < 1e-2


# -- convolved projections -----------------------------------------------------------------------------------------------------
class Convolved:
    """Projected rows of sequences, fed in portions; queries, cache and handed-on values against the whole sequences at once."""

    def __init__(self, H, G, D, vdim, taps, lens, rot, seed=0):
        self.H, self.G, self.D, self.vdim, self.lens, self.rot = H, G, D, vdim, lens, rot
        self.cols, self.pages = (H + 2 * G) * D, [-(-n // 64) for n in lens]
        self.u = [rnd(n, self.cols, seed=seed + i) for i, n in enumerate(lens)]
        for x in self.u:
            x.view(-1, H + 2 * G, D)[:, H + G:, vdim:] = 0                  # what padding holds
        self.taps, self.gain, self.share = rnd(taps, self.cols, seed=seed + 50), 1 + rnd(H, seed=seed + 51, scale=0.3), torch.tensor([0.3], device="cuda")
        self.first = [rnd(n, G, vdim, seed=seed + 60 + i) for i, n in enumerate(lens)]
        self.slots = torch.randperm(len(lens) + 2, generator=torch.Generator().manual_seed(seed))[:len(lens)].tolist()
        order = torch.randperm(sum(self.pages), generator=torch.Generator().manual_seed(seed + 1)).add(1).tolist()
        at = [sum(self.pages[:i]) for i in range(len(lens))]
        self.table = ints([(order[a:a + n] + [0] * max(self.pages))[:max(self.pages)] for a, n in zip(at, self.pages)])
        self.ring = torch.full((len(lens) + 2, taps, self.cols), float("nan"), device="cuda")      # what a former owner left

    def run(self, cuts, dtype, decode_f32, mode):
        """``cuts``: portion sizes (the last repeats); portions of one row in all sequences are decode steps."""
        from llaminar_b200.ops import grouped as ops
        kv = torch.zeros(sum(self.pages) + 1, 2, self.G, 64, self.D, dtype=dtype, device="cuda")
        q = [torch.zeros(n, self.H, self.D, device="cuda") for n in self.lens]
        kept = [torch.zeros(n, self.G, self.vdim, device="cuda") for n in self.lens]
        half = self.rot["dims"] // 2
        freqs, grow = oracle.yarn(self.rot)
        done, i = [0] * len(self.lens), 0
        while any(d < n for d, n in zip(done, self.lens)):
            size = cuts[min(i, len(cuts) - 1)]
            live = [b for b, n in enumerate(self.lens) if done[b] < n]
            part = {b: min(size, self.lens[b] - done[b]) for b in live}
            decode = all(n == 1 for n in part.values())
            rows = torch.cat([self.u[b][done[b]:done[b] + part[b]] for b in live]).to(F32 if dtype == F32 or (decode and decode_f32) else dtype)
            pos = [p for b in live for p in range(done[b], done[b] + part[b])]
            ang = torch.tensor([[p * f for f in freqs] for p in pos], dtype=F64)
            ang = (torch.stack([ang.cos(), ang.sin()], -1) * grow).float().cuda().view(-1, half, 2)
            first = torch.cat([self.first[b][done[b]:done[b] + part[b]] for b in live]).contiguous() if mode == "mix" else torch.zeros(len(pos), self.G, self.vdim, device="cuda")
            out = torch.empty(len(pos), self.H, self.D, dtype=dtype, device="cuda")
            cu = [0]
            for b in live:
                cu.append(cu[-1] + part[b])
            ops.conv_prep(rows, self.taps, self.ring, ints([self.slots[b] for b in live]), None if decode else ints(cu), ang, self.gain, first if mode != "none" else None,
                          self.share if mode == "mix" else None, ints(pos), ints([k for k, b in enumerate(live) for _ in range(part[b])]), self.table[live].contiguous(), out, kv)
            for k, b in enumerate(live):
                q[b][done[b]:done[b] + part[b]] = out[cu[k]:cu[k + 1]].float()
                kept[b][done[b]:done[b] + part[b]] = first[cu[k]:cu[k + 1]]
                done[b] += part[b]
            i += 1
        return q, kv, kept

    def check(self, got, mode, tol):
        q, kv, kept = got
        for b, n in enumerate(self.lens):
            y = oracle.short_conv(self.u[b].double().cpu(), self.taps.double().cpu().T).view(n, -1, self.D)
            turn = lambda x: oracle.rotate_halves(x.transpose(0, 1), range(n), self.rot).transpose(0, 1)
            v = y[:, self.H + self.G:, :self.vdim]
            if mode == "first":
                assert err(kept[b], v) < tol
            if mode == "mix":
                v = oracle.mix_values(v, self.first[b].double().cpu(), self.share.double().cpu())
            page, off = self.table[b][torch.arange(n) // 64].long(), torch.arange(n) % 64
            assert err(q[b], turn(y[:, :self.H]) * self.gain.double().cpu()[:, None]) < tol
            assert err(kv[page, 0, :, off], turn(y[:, self.H:self.H + self.G])) < tol
            assert err(kv[page, 1, :, off][..., :self.vdim], v) < tol and bool((kv[page, 1, :, off][..., self.vdim:] == 0).all())


YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}


@both
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("mode", ["none", "first", "mix"])
def test_conv_prep(taps, mode, dtype):
    """Whole prompts (short ones and ones long enough for strips of rows), portions of every size, decode steps; slots hold junk first."""
    for H, G, D, vdim, lens, rot in ((5, 2, 64, 40, [70, 3, 130, 1], 32), (6, 3, 128, 128, [400, 7, 300], 128), (2, 1, 136, 72, [30, 9], 20)):
        x = Convolved(H, G, D, vdim, taps, lens, {"dims": rot, "base": 100.0, "scaling": YARN})
        for cuts in ([500], [1], [2], [5, 1, 3, 60], [64, 66, 1]):
            x.ring.fill_(float("nan"))
            x.check(x.run(cuts, dtype, True, mode), mode, 2e-2 if dtype == BF else 1e-5)


# -- lightning attention -------------------------------------------------------------------------------------------------------
def gated(o, z, w, true_n):
    n = o.shape[0]
    o = o.reshape(n, -1)
    return o / torch.sqrt((o * o).sum(-1, keepdim=True) / true_n + EPS) * w * torch.sigmoid(z)


@both
@pytest.mark.parametrize("heads,dim,vdim,decay", [(3, 64, 32, (0.6, 0.99, 1.0)), (2, 128, 256, (0.999, 0.5)), (1, 24, 320, (0.97,)), (5, 8, 8, (0.0, 0.1, 0.3, 0.9, 0.998))])
def test_lightning(heads, dim, vdim, decay, dtype):
    """Sequences of unequal lengths in portions, row by row and chunk by chunk; slots hold junk before a sequence starts."""
    from llaminar_b200.ops import dense, mixers
    lens = [300, 5, 129, 128, 1]
    n_qkv, nv = 2 * heads * dim + heads * vdim, heads * vdim
    u = [rnd(n, n_qkv + nv, seed=i).to(dtype) for i, n in enumerate(lens)]
    w, dec = 1 + rnd(nv, seed=20, scale=0.3), torch.tensor(decay, device="cuda")
    offs = [0, heads * dim, 2 * heads * dim, n_qkv]
    want, state = [], []
    for x in u:
        x = x.double().cpu()
        q, k, v = (oracle.silu(x[:, a:a + heads * s]).view(-1, heads, s) for a, s in zip(offs, (dim, dim, vdim)))
        want.append(gated(oracle.decayed_state(q, k, v, dec.double().cpu()), x[:, n_qkv:], w.double().cpu(), nv))
        S = torch.zeros(heads, dim, vdim, dtype=F64)
        for t in range(len(x)):
            S = dec.double().cpu()[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        state.append(S.transpose(1, 2))
    tol = 3e-2 if dtype == BF else 1e-5
    for chunked in ([False, True] if dtype == BF else [False]):
        S = torch.full((len(lens) + 1, heads, vdim, dim), 7.0, device="cuda")
        slots, done, got = [3, 0, 5, 1, 4], [0] * len(lens), [[] for _ in lens]
        for size in (130, 1, 40, 500):
            live = [b for b, n in enumerate(lens) if done[b] < n]
            part = [min(size, lens[b] - done[b]) for b in live]
            decode = not chunked and all(n == 1 for n in part)
            rows = torch.cat([u[b][done[b]:done[b] + n] for b, n in zip(live, part)])
            if decode:
                rows = rows.float()
            cu = [sum(part[:i]) for i in range(len(part) + 1)]
            pos = ints([p for b, n in zip(live, part) for p in range(done[b], done[b] + n)])
            raw, out = torch.empty(len(rows), nv, dtype=rows.dtype, device="cuda"), torch.empty(len(rows), nv, dtype=dtype, device="cuda")
            args = (rows, offs, None, dec, None, 1.0, 1.0, None if decode else ints(cu), pos, ints([slots[b] for b in live]), (S,), vdim, None, False)
            if chunked:
                dense.activate(rows[:, :n_qkv], rows[:, :n_qkv], dense.ACT_SILU)
                mixers.linear_chunk(*args, out, EPS, mixers.chunk_tables(cu, "cuda"), raw, status(), only_raw=True)
                assert int(status()[0]) == 0
            else:
                mixers.linear_rows(*args, raw, EPS, silu_in=True, raw=True)
            mixers.joint_gate(raw, rows, n_qkv, w, nv, out, EPS)
            for i, b in enumerate(live):
                got[b].append(out[cu[i]:cu[i + 1]])
                done[b] += part[i]
        for b in range(len(lens)):
            assert err(torch.cat(got[b]), want[b]) < tol, (chunked, b, err(torch.cat(got[b]), want[b]))
            assert err(S[slots[b]], state[b]) < (1e-2 if dtype == BF else 1e-5)
        assert bool((S[2] == 7).all())                                              # nobody's slot


@both
@pytest.mark.parametrize("n,true_n", [(64, 64), (4096, 4096), (6000, 5990), (40, 33)])
def test_joint_gate(n, true_n, dtype):
    from llaminar_b200.ops import mixers
    o, rows, w, out = rnd(9, n, seed=1).to(dtype), rnd(9, n + 16, seed=2).to(dtype), rnd(n, seed=3), torch.empty(9, n, dtype=dtype, device="cuda")
    o[:, true_n:] = 0
    mixers.joint_gate(o, rows, 16, w, true_n, out, EPS)
    assert err(out, gated(o.double(), rows[:, 16:].double(), w.double(), true_n)) < (1e-2 if dtype == BF else 1e-5)


# -- experts -------------------------------------------------------------------------------------------------------------------
@both
@pytest.mark.parametrize("E,top,groups,keep", [(8, 3, 4, 2), (6, 2, 2, 1), (40, 5, 40, 9), (128, 8, 8, 4), (300, 4, 100, 7), (1000, 6, 500, 3), (5, 5, 1, 1), (33, 2, 3, 1)])
def test_grouped_routing(E, top, groups, keep, dtype):
    from llaminar_b200.ops import experts as ops
    router = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}}
    for T in (3, 70):
        x, r = rnd(T, 72, seed=T).to(dtype), rnd(E, 72, seed=1, scale=0.4).to(dtype)
        W = lambda name: r.double().cpu()
        ids, wt = oracle.route(x.double().cpu(), W, router)
        clear = oracle.router_gap(x.double().cpu(), W, router) > 1e-4
        assert clear.float().mean() > 0.8
        for form in ("x", "logits"):
            got, w = torch.full((T, top), -1, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
            kw = dict(x=x, router=r) if form == "x" else dict(logits=x.float() @ r.float().T)
            ops.expert_route(None, got, w, **kw, groups=groups, keep=keep)
            a, b = got.cpu().long().sort(-1), ids.sort(-1)
            assert torch.equal(a.values[clear], b.values[clear])
            assert (w.double().cpu().gather(1, a.indices) - wt.gather(1, b.indices))[clear].abs().max() < 1e-5


def test_grouped_routing_of_equal_and_broken_logits():
    from llaminar_b200.ops import experts as ops
    ids, w = torch.empty(4, 4, dtype=torch.int32, device="cuda"), torch.empty(4, 4, device="cuda")
    z = torch.zeros(4, 12, device="cuda")
    z[1], z[2], z[3] = float("nan"), float("-inf"), -float("nan")
    ops.expert_route(None, ids, w, logits=z, groups=4, keep=2)
    assert ids[0].tolist() == [0, 1, 2, 3] and torch.allclose(w[0], torch.full((4,), 0.25, device="cuda"))
    assert bool(((ids >= 0) & (ids < 12)).all())


@pytest.mark.parametrize("T,E,top,d,ff", [(1, 8, 2, 256, 104), (9, 6, 3, 200, 72), (300, 5, 2, 136, 264)])
def test_limited_experts(T, E, top, d, ff):
    """All three forms of the product; the limits bind on a good part of the values."""
    from llaminar_b200.ops import experts as ops
    limit, P = 0.7, T * top
    x, gu = rnd(T, d).bfloat16(), rnd(E, 2 * ff, d, seed=1, scale=d ** -0.5).bfloat16()
    ids = torch.randint(0, E, (T, top), generator=torch.Generator().manual_seed(2)).int().cuda()
    eye = torch.eye(ff, dtype=F64, device="cuda")
    want = torch.cat([oracle.limited_ffn(x[p // top].double()[None], lambda n: {"gate": gu[e, :ff].double(), "up": gu[e, ff:].double(), "down": eye}[n], limit)
                      for p, e in enumerate(ids.view(-1).tolist())])
    out = torch.empty(P, ff, dtype=BF, device="cuda")
    if P <= ops.max_pairs():
        ops.expert_rows(gu, x, ids, out, top, True, limit)
        assert err(out, want) < 1e-2
    out32 = torch.empty(P, ff, device="cuda")
    ops.expert_plain(gu.float(), x.float(), ids, out32, top, True, limit)
    assert err(out32, want) < 1e-5
    order = ids.view(-1).long().argsort(stable=True)
    counts = torch.bincount(ids.view(-1).long(), minlength=E).int()
    ops.expert_grouped(gu, x[order // top].contiguous(), counts, out, True, status(), limit)
    assert int(status()[0]) == 0 and err(out, want[order]) < 1e-2
