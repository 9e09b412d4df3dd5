"""Throughput and kernel times of models with recurrent mixers (zogepel) beside the like parts of the other families at equal size.

Used by `bench.py --mixers`.  Two parts: whole models (prefill and decode tokens per second through the engine, random weights, a
few layers of full size) and single kernels with their fraction of the memory or tensor roofline.  The like kernels: Gated-DeltaNet
for the recurrences (a state of the same size), grouped-query attention of qwen3-8b, norms and products of pozivik-8b and qwen3-8b.
"""
from __future__ import annotations

import json

import torch

from .bench_util import copies_for, cut, measured_peaks, page_tables, row, time_us, visible_pairs, whole_model
from .models.config import SHAPES, MatrixLSTM, ModelConfig, ParallelMixers

BF = dict(dtype=torch.bfloat16, device="cuda")
F32 = dict(dtype=torch.float32, device="cuda")


def _int(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


class Linear:
    """One recurrent mixer with random rows and `slots` state slots."""

    def __init__(self, m, rows: int, slots: int, dtype, copies: int, state_copies: int):
        self.m, H, d, v = m, m.heads, m.dim, m.vdim
        self.lstm = isinstance(m, MatrixLSTM)
        self.offs = [0, H * d, 2 * H * d, 2 * H * d + H * v]
        self.rows = [torch.randn(rows, 2 * H * (d + v), dtype=dtype, device="cuda") for _ in range(copies)]
        self.gates = (torch.randn(rows, 2 * H, **F32), torch.zeros(H, **F32), torch.full((H,), 4.0, **F32), m.gate_cap) if self.lstm else None
        self.decay = None if self.lstm else torch.tensor(m.decay, **F32)
        self.angles = None if self.lstm else torch.rand(rows, m.rotary.dims // 2, 2, **F32)
        self.norm = torch.ones(H * v, **F32) if self.lstm else None
        shapes = [(slots + 1, H, v, d)] + ([(slots + 1, H, d), (slots + 1, H)] if self.lstm else [])
        self.states = [tuple(torch.zeros(*s, **F32) for s in shapes) for _ in range(state_copies)]
        self.out = [torch.empty(rows, H * v, **BF) for _ in range(copies)]
        self.name = "mLSTM" if self.lstm else "retention"

    def args(self, i: int, cu, positions, slots):
        n = len(self.rows)
        return (self.rows[i % n], self.offs, self.gates, self.decay, self.angles, 1.0 if not self.lstm else self.m.dim ** -0.5,
                self.m.dim ** -0.5 if not self.lstm else 1.0, cu, positions, slots, self.states[i % len(self.states)], self.m.vdim, self.norm,
                not self.lstm, self.out[i % n], 1e-5)


def linear_decode(m, batch: int) -> dict:
    from .ops import mixers as ops
    nbytes = batch * 2 * m.heads * m.dim * m.vdim * 4
    k = copies_for(nbytes)
    x = Linear(m, batch, batch, torch.float32, 1, k)
    pos, slots = torch.full((batch,), 500, dtype=torch.int32, device="cuda"), torch.arange(batch, dtype=torch.int32, device="cuda")
    us = time_us([lambda i=i: ops.linear_rows(*x.args(i, None, pos, slots)) for i in range(k)])
    return row(f"linear_rows {x.name} batch {batch} heads {m.heads} x {m.dim} x {m.vdim}", us, nbytes + 4 * x.rows[0].numel(), 0)


def gdn_decode(batch: int, heads: int, d: int) -> dict:
    """Gated-DeltaNet step with the same number of state values."""
    from . import ops
    nbytes = batch * 2 * heads * d * d * 4
    k = copies_for(nbytes)
    C = 3 * heads * d
    recs = [torch.zeros(batch + 1, heads, d, d, **F32) for _ in range(k)]
    inp, conv = torch.randn(batch, C + heads * d + 2 * heads, **BF), torch.zeros(batch + 1, C, 3, **F32)
    w, v = torch.randn(C, 4, **F32), torch.zeros(heads, **F32)
    y, out, slots = torch.empty(batch, C, **F32), torch.empty(batch, heads * d, **BF), torch.arange(batch, dtype=torch.int32, device="cuda")
    us = time_us([lambda r=r: ops.gdn_step(inp, C, C, C + heads * d, w, v - 1, v, torch.ones(d, **F32), conv, r, slots, y, out, heads, 0, 1e-6) for r in recs])
    return row(f"gdn_step batch {batch} heads {heads} x {d} x {d} (hybrid family)", us, nbytes + batch * C * 12 * 2, 0)


def linear_prefill(m, n: int) -> dict:
    """All of the chunk-parallel form: chunk sums, scan, outputs, norm and gate."""
    from . import ops as base
    from .ops import mixers as ops
    copies = 3
    x = Linear(m, n, 1, torch.bfloat16, copies, copies)
    cu, pos, slots = _int([0, n]), torch.arange(n, dtype=torch.int32, device="cuda"), _int([0])
    tables, raw = ops.chunk_tables([0, n], "cuda"), torch.empty(n, m.heads * m.vdim, **BF)
    status = base.scratch_for(torch.device("cuda", torch.cuda.current_device())).status
    us = time_us([lambda i=i: ops.linear_chunk(*x.args(i, cu, pos, slots), tables, raw, status) for i in range(copies)] * 2)
    assert int(status[0]) == 0
    C = 128
    flops = 2.0 * n * m.heads * (C / 2 * (m.dim + m.vdim) + 2 * m.dim * m.vdim)
    return row(f"linear_chunk {x.name} rows {n} heads {m.heads} x {m.dim} x {m.vdim} (three launches)", us, 2.0 * n * m.heads * (2 * m.dim + 3 * m.vdim), flops)


def gdn_prefill(n: int, heads: int, d: int) -> dict:
    from .models import gdn
    C = 3 * heads * d
    qkv, z, ab = torch.randn(n, C, **F32), torch.randn(n, heads * d, **F32), torch.randn(2, n, heads, **F32)
    conv, rec = torch.zeros(1, C, 3, **F32), torch.zeros(1, heads, d, d, **F32)
    w, v, o = torch.randn(C, 4, **F32), torch.zeros(heads, **F32), torch.ones(d, **F32)
    call = lambda: gdn.gdn_block_rows(qkv, z, ab[0], ab[1], [(0, n, 0, True)], conv, rec, w, v - 1, v, o, heads, heads, d, 1e-6)
    call()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    call()
    b.record()
    torch.cuda.synchronize()
    return row(f"gdn prefill rows {n} heads {heads} x {d} x {d} (hybrid family, PyTorch ops)", a.elapsed_time(b) * 1e3, 2.0 * n * heads * d * 5, 2.0 * n * heads * (64 * d + 3 * d * d))


def attention(cfg: ModelConfig, gqa: ModelConfig) -> list[dict]:
    from . import ops as base
    from .ops import grouped as ops
    m = next(x.left for x in cfg.mixers if isinstance(x, ParallelMixers))
    H, G, D, sc = m.heads, m.kv_heads, m.dim, base.scratch_for(torch.device("cuda", torch.cuda.current_device()))
    sink, out = torch.zeros(H, **F32), []
    for batch, ctx in ((1, 2048), (32, 2048)):
        bt, P, pages = page_tables(batch, ctx, "cuda")
        keys = min(ctx, m.window)
        nbytes = batch * keys * 2 * G * D * 2
        kvs = [torch.randn(pages, 2, G, 64, D, **BF) for _ in range(copies_for(nbytes))]
        q, o, gate = torch.randn(batch, H, D, **BF), torch.empty(batch, H * D, **BF), torch.randn(batch, H * D, **F32)
        lens, sp = torch.full((batch,), ctx, dtype=torch.int32, device="cuda"), ops.decode_splits(batch, G, D, P, m.window, sc)
        us = time_us([lambda kv=kv: ops.attn_decode(q, kv, o, bt, lens, m.scale, sp, m.window, sink, gate, sc) for kv in kvs])
        out.append(row(f"attn_decode window {m.window} sinks gate batch {batch} heads {H}/{G}", us, nbytes + 8 * q.numel(), 4.0 * batch * H * keys * D))
        bt, P, pages = page_tables(batch, keys, "cuda")
        kvs = [torch.randn(pages, 2, G, 64, D, **BF) for _ in range(copies_for(nbytes))]
        lens, sp = torch.full((batch,), keys, dtype=torch.int32, device="cuda"), max(1, min(16, 296 // (batch * G), P // 2))
        us = time_us([lambda kv=kv: base.attn_decode(q, kv, o, bt, lens, H, G, D, 1, m.scale, sp, sc) for kv in kvs])
        out.append(row(f"attn_decode keys {keys} batch {batch} heads {H}/{G} (qwen3-8b)", us, nbytes + 4 * q.numel(), 4.0 * batch * H * keys * D))
        del kvs
    for n in (1024, 4096):
        bt, P, pages = page_tables(1, n, "cuda")
        cols = (2 * H + G) * D
        rows = [torch.randn(n, cols, **BF) for _ in range(3)]
        qs, kvs, o = [torch.randn(n, H, D, **BF) for _ in range(3)], [torch.randn(pages, 2, G, 64, D, **BF) for _ in range(3)], torch.empty(n, H * D, **BF)
        cu, ctx = _int([0, n]), _int([0])
        for window in (m.window, 0):
            us = time_us([lambda i=i: ops.attn_prefill(qs[i], kvs[i], o, bt, cu, ctx, m.scale, n, window, sink, rows[i][:, cols - H * D:], sc.status) for i in range(3)] * 3)
            out.append(row(f"attn_prefill sinks gate rows {n} window {window or 'none'} heads {H}/{G}", us, 2.0 * n * (3 * H + 2 * G) * D, 4.0 * visible_pairs(n, window) * H * D))
        us = time_us([lambda i=i: base.attn_prefill(qs[i], kvs[i], o, bt, cu, ctx, H, G, D, m.scale, n, scratch=sc) for i in range(3)] * 3)
        out.append(row(f"attn_prefill rows {n} heads {H}/{G} (qwen3-8b)", us, 2.0 * n * (2 * H + 2 * G) * D, 4.0 * visible_pairs(n, 0) * H * D))
        assert int(sc.status[0]) == 0
    for n in (32, 4096):
        bt, P, pages = page_tables(1, n, "cuda")
        cols, k = (H + G) * D, 24 if n > 100 else 256
        rows, q, kv = [torch.randn(n, cols, **BF) for _ in range(k)], torch.empty(n, H, D, **BF), torch.zeros(pages, 2, G, 64, D, **BF)
        pos, sid = torch.arange(n, dtype=torch.int32, device="cuda"), torch.zeros(n, dtype=torch.int32, device="cuda")
        qn, kn = torch.ones(H * D, **F32), torch.ones(G * D, **F32)
        us = time_us([lambda r=r: ops.attn_prep(r, 0, H * D, H * D, qn, kn, pos, sid, bt, q, kv, D, 1e-5) for r in rows])
        out.append(row(f"attn_prep rows {n}", us, 2.0 * n * D * (2 * H + 3 * G), 0))
        rows = [torch.randn(n, (H + 2 * G) * D, **BF) for _ in range(k)]
        us = time_us([lambda r=r: base.rope_kv(r, q, kv, qn[:D], kn[:D], pos, sid, bt, H, G, D, 1e6, 1e-6) for r in rows])
        out.append(row(f"rope_kv rows {n} (qwen3-8b)", us, 2.0 * n * D * (2 * H + 4 * G), 0))
    return out


def row_wise(cfg: ModelConfig, n: int) -> list[dict]:
    """Residual updates and activations, beside pozivik's."""
    from .ops import dense as ops
    d, ff, sd = cfg.d_model, cfg.ff_width(0), cfg.side_dim
    w, k = torch.ones(d, **F32), min(copies_for(n * d * 12), 64)
    hs, ys, y2, xs = [torch.randn(n, d, **F32) for _ in range(k)], [torch.randn(n, d, **BF) for _ in range(k)], [torch.randn(n, d, **BF) for _ in range(k)], [torch.empty(n, d, **BF) for _ in range(k)]
    out = [row(f"resid_norm rows {n} (layer norm, residual update, copy)", time_us([lambda h=h, y=y, x=x: ops.resid_norm(h, y, w, copy0=x, center_post=True, eps=1e-6) for h, y, x in zip(hs, ys, xs)]), n * d * 12, 0),
           row(f"resid_norm rows {n} (two sides)", time_us([lambda h=h, y=y, z=z, x=x: ops.resid_norm(h, y, w, y2=z, w_y=w, w_y2=w, copy0=x, center_post=True, eps=1e-6) for h, y, z, x in zip(hs, ys, y2, xs)]), n * d * 14, 0),
           row(f"resid_norm rows {n} (pozivik: two norms)", time_us([lambda h=h, y=y, x=x: ops.resid_norm(h, y, w, w_next=w, xn=x, eps=1e-6) for h, y, x in zip(hs, ys, xs)]), n * d * 12, 0)]
    k = min(copies_for(n * ff * 4), 64)
    raw, act = [torch.randn(n, 2 * ff, **BF) for _ in range(k)], torch.empty(n, ff, **BF)
    half = [r.view(2 * n, ff)[:n] for r in raw]
    out.append(row(f"activate relu2 rows {n}", time_us([lambda r=r: ops.activate(r, act, ops.ACT_RELU2) for r in half]), n * ff * 4, 0))
    out.append(row(f"activate gelu_mul rows {n} (pozivik)", time_us([lambda r=r: ops.activate(r, act, ops.ACT_GELU_MUL) for r in raw]), n * ff * 6, 0))
    table, tok = torch.randn(4096, 36 * sd, **BF), torch.randint(0, 4096, (n,), dtype=torch.int32, device="cuda")
    ks = min(copies_for(n * sd * 6), 256)
    gs, act = [torch.randn(n, sd, **BF) for _ in range(ks)], torch.empty(n, sd, **BF)
    out.append(row(f"activate gelu_side rows {n} width {sd}", time_us([lambda i=i, g=g: ops.activate(g, act, ops.ACT_GELU_SIDE, (table, i % 36 * sd, sd, tok)) for i, g in enumerate(gs)]), n * sd * 6, 0))
    return out


def products(cfg: ModelConfig, rows_list=(1, 8, 32)) -> list[dict]:
    from .engine.dense import DenseLinear
    from .ops import dense as ops
    d, ff, sd = cfg.d_model, cfg.ff_width(0), cfg.side_dim
    m, par = cfg.mixers[0], next(x for x in cfg.mixers if isinstance(x, ParallelMixers))
    lin = lambda r: 2 * r.heads * (r.dim + r.vdim)
    shapes = {"mLSTM in": (lin(m), d), "gates": (2 * m.heads, d), "parallel in": ((2 * par.left.heads + par.left.kv_heads) * par.left.dim + lin(par.right), d),
              "out": (d, m.heads * m.vdim), "down": (d, ff), "side_proj": (d, sd)}
    out = []
    for rows in rows_list:
        for name, (n, k) in shapes.items():
            c = copies_for(n * k * 2)
            lins, x = [DenseLinear(torch.randn(n, k, **BF)) for _ in range(c)], torch.randn(rows, k, **BF)
            y = torch.empty(rows, n, **(F32 if " in" in name or name == "gates" else BF))
            out.append(row(f"{name} [{n}, {k}] x {rows} rows", time_us([lambda l=l: l(x, y) for l in lins]), n * k * 2, 2.0 * n * k * rows))
            del lins
        c = copies_for(ff * d * 2)
        lins, x = [DenseLinear(torch.randn(ff, d, **BF)) for _ in range(c)], torch.randn(rows, d, **BF)
        act, raw = torch.empty(rows, ff, **BF), torch.empty(rows, ff, **BF)
        out.append(row(f"up + relu2 [{ff}, {d}] x {rows} rows", time_us([lambda l=l: l.activated(x, act, raw, ops.ACT_RELU2) for l in lins]), ff * d * 2, 2.0 * ff * d * rows))
        lins = [DenseLinear(torch.randn(2 * ff, d, **BF)) for _ in range(c)]
        gu = torch.empty(rows, 2 * ff, **BF)
        out.append(row(f"gate|up + gelu [{2 * ff}, {d}] x {rows} rows (pozivik)", time_us([lambda l=l: l.gelu(x, act, gu) for l in lins]), ff * d * 4, 4.0 * ff * d * rows))
        del lins
        table, tok = torch.randn(4096, 36 * sd, **BF), torch.randint(0, 4096, (rows,), dtype=torch.int32, device="cuda")
        lins, act, raw = [DenseLinear(torch.randn(sd, d, **BF)) for _ in range(128)], torch.empty(rows, sd, **BF), torch.empty(rows, sd, **BF)
        out.append(row(f"side_gate + gelu [{sd}, {d}] x {rows} rows", time_us([lambda l=l: l.activated(x, act, raw, ops.ACT_GELU_SIDE, (table, 0, sd, tok)) for l in lins]), sd * d * 2, 2.0 * sd * d * rows))
        del lins
    return out


def run(layers: int = 8, log=print) -> dict:
    cfg, gqa, lat = SHAPES["zogepel-8b"], SHAPES["qwen3-8b"], SHAPES["pozivik-8b"]
    lstm, ret = cfg.mixers[0], cfg.mixers[1].right
    kernels = []
    for batch in (1, 8, 32, 128):
        kernels += [linear_decode(lstm, batch), linear_decode(ret, batch), gdn_decode(batch, lstm.heads * lstm.vdim // lstm.dim, lstm.dim)]
    for n in (1024, 4096, 8192):
        kernels += [linear_prefill(lstm, n), linear_prefill(ret, n), gdn_prefill(n, lstm.heads * lstm.vdim // lstm.dim, lstm.dim)]
    kernels += attention(cfg, gqa)
    for n in (32, 4096):
        kernels += row_wise(cfg, n)
    kernels += products(cfg)
    for k in kernels:
        log(json.dumps(k))
    models = []
    for batch, prompt in ((1, 2048), (32, 1024)):
        for c in (cfg, lat, gqa):
            models.append(whole_model(cut(c, layers), "BF16", prompt, batch))
            log(json.dumps(models[-1]))
    return {"peaks": measured_peaks()[2], "l2": "inputs larger than L2", "kernels": kernels, "models": models}
