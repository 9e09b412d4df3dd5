"""Throughput and kernel times of latent-attention models beside the like parts of a grouped-query model of equal size.

Used by `bench.py --latent`.  Two parts: whole models (prefill and decode tokens per second through the engine, random
weights, a few layers of full size) and single kernels with their fraction of the memory or tensor roofline.
"""
from __future__ import annotations

import json
from dataclasses import replace

import torch

from .bench_util import copies_for, cut, measured_peaks, page_tables, row, time_us, visible_pairs, whole_model
from .models.config import SHAPES, ModelConfig

def latent_decode(cfg: ModelConfig, batch: int, ctx: int, tensor_core: bool = True) -> dict:
    """One layer's attention of a decode step: query rotation, split attention and merge."""
    from .ops import latent as ops
    from .engine.latent import PART_FLOATS, PaddedSizes
    m, dev = cfg.mixers[0], "cuda"
    s = PaddedSizes.of(m)
    bt, P, pages = page_tables(batch, ctx, dev)
    keys = min(ctx, m.window) if m.window else ctx
    nbytes = batch * keys * s.width * 2
    bf = dict(dtype=torch.bfloat16, device=dev)
    kvs = [torch.randn(pages, 64, s.width, **bf) for _ in range(copies_for(nbytes))]
    q, ql = torch.randn(batch, s.heads, s.dim + s.rot, **bf), torch.randn(s.heads, batch, s.latent, **bf)
    out = torch.empty_like(ql)
    pos = torch.full((batch,), ctx - 1, dtype=torch.int32, device=dev)
    sid = torch.arange(batch, dtype=torch.int32, device=dev)
    ang = torch.rand(batch, m.rotary.dims // 2, 2, device=dev)
    sink = torch.zeros(s.heads, device=dev)
    po, pm = torch.empty(PART_FLOATS, device=dev), torch.empty(PART_FLOATS // 4, device=dev)
    group = ops.rows_group(kvs[0], s.latent, m.rot_dim, s.heads, tensor_core)
    sp = ops.rows_splits(batch, s.heads, group, tensor_core, min(P * 64, m.window) if m.window else P * 64, s.latent, PART_FLOATS)
    status = torch.zeros(4, dtype=torch.int32, device=dev)
    calls = [lambda kv=kv: ops.latent_rows(ql, q, s.dim, ang, None, pos, sid, bt, kv, m.rot_dim, m.window, m.scale, sink, out, po, pm, sp, group, status) for kv in kvs]
    us = time_us(calls)
    assert int(status[0]) == 0
    flops = 2.0 * batch * s.heads * keys * (s.width + s.latent)
    return row(f"latent_rows ({'tcgen05' if tensor_core else 'mma.sync'}) batch {batch} keys {keys} heads {s.heads} splits {sp}", us, nbytes + 4 * ql.numel(), flops)


def gqa_decode(cfg: ModelConfig, batch: int, ctx: int) -> dict:
    from . import ops
    dev, H, Hk, D = "cuda", cfg.n_heads, cfg.n_kv_heads, cfg.head_dim
    bt, P, pages = page_tables(batch, ctx, dev)
    nbytes = batch * ctx * 2 * Hk * D * 2
    bf = dict(dtype=torch.bfloat16, device=dev)
    kvs = [torch.randn(pages, 2, Hk, 64, D, **bf) for _ in range(copies_for(nbytes))]
    q = torch.randn(batch, H, D, **bf)
    out, lens = torch.empty_like(q), torch.full((batch,), ctx, dtype=torch.int32, device=dev)
    sp = max(1, min(16, 296 // max(1, batch * Hk), P // 2))
    sc = ops.scratch_for(torch.device("cuda", torch.cuda.current_device()))
    us = time_us([lambda kv=kv: ops.attn_decode(q, kv, out, bt, lens, H, Hk, D, 1, D ** -0.5, sp, sc) for kv in kvs])
    return row(f"attn_decode batch {batch} keys {ctx} heads {H}/{Hk}", us, nbytes + 4 * q.numel(), 4.0 * batch * H * ctx * D)


def latent_prefill(cfg: ModelConfig, n: int, window: int) -> list[dict]:
    """One layer's prompt attention: the attention kernel, and the key/value expansion before it."""
    from .ops import latent as ops
    from .engine.latent import PaddedSizes
    m, dev = replace(cfg.mixers[0], window=window), "cuda"
    s = PaddedSizes.of(m)
    bt, P, pages = page_tables(1, n, dev)
    bf = dict(dtype=torch.bfloat16, device=dev)
    copies = 3
    q = [torch.randn(n, s.heads, s.dim + s.rot, **bf) for _ in range(copies)]
    ks, vs = [torch.randn(n, s.heads * s.dim, **bf) for _ in range(copies)], [torch.randn(n, s.heads * s.vdim, **bf) for _ in range(copies)]
    vts = [torch.randn(s.heads * s.vdim, n, **bf) for _ in range(copies)]
    lat, out = torch.randn(n, s.width, **bf), torch.empty(n, s.heads * s.vdim, **bf)
    kv = torch.randn(pages, 64, s.width, **bf)
    ang, sink = torch.rand(n, m.rotary.dims // 2, 2, device=dev), torch.zeros(s.heads, device=dev)
    seqs = torch.tensor([[0, 0, n, 0, 0, 0, n, 0]], dtype=torch.int32, device=dev)
    wk, wv = torch.randn(s.heads * s.dim, s.latent, **bf), torch.randn(s.heads * s.vdim, s.latent, **bf)
    status = torch.zeros(4, dtype=torch.int32, device=dev)
    pairs, rows = visible_pairs(n, window), []
    for name, v, st in (("tcgen05", vts, status), ("mma.sync", vs, None)):
        us = time_us([lambda i=i: ops.latent_chunk(q[i], ang, ks[i], v[i], lat, s.latent, seqs, n, out, s.dim, s.rot, s.vdim, window, m.scale, sink, st) for i in range(copies)] * 3)
        rows.append(row(f"latent_chunk ({name}) rows {n} window {window or 'none'} heads {s.heads}", us, 2 * (q[0].numel() + 3 * ks[0].numel()),
                         2.0 * pairs * s.heads * (m.dim + m.rot_dim + m.vdim)))
    assert int(status[0]) == 0
    c = lat[:, :s.latent]
    us = time_us([lambda i=i: (torch.mm(c, wk.t(), out=ks[i]), torch.mm(wv, c.t(), out=vts[i])) for i in range(copies)] * 3)
    rows.append(row(f"keys and values from latents (two cuBLAS products) rows {n}", us, 2 * (2 * ks[0].numel() + lat.numel()), 2.0 * n * (wk.numel() + wv.numel())))
    lats = [torch.empty_like(lat) for _ in range(copies_for(4 * lat.numel()))]
    us = time_us([lambda l=l: ops.latent_gather(kv, seqs, n, bt, l) for l in lats])
    rows.append(row(f"latent_gather rows {n}", us, 4 * lat.numel(), 0))
    return rows


def gqa_prefill(cfg: ModelConfig, n: int) -> dict:
    from . import ops
    dev, H, Hk, D = "cuda", cfg.n_heads, cfg.n_kv_heads, cfg.head_dim
    bt, P, pages = page_tables(1, n, dev)
    bf = dict(dtype=torch.bfloat16, device=dev)
    qs = [torch.randn(n, H, D, **bf) for _ in range(3)]
    kvs = [torch.randn(pages, 2, Hk, 64, D, **bf) for _ in range(3)]
    out = torch.empty_like(qs[0])
    cu, ctx = torch.tensor([0, n], dtype=torch.int32, device=dev), torch.zeros(1, dtype=torch.int32, device=dev)
    sc = ops.scratch_for(torch.device("cuda", torch.cuda.current_device()))
    us = time_us([lambda q=q, kv=kv: ops.attn_prefill(q, kv, out, bt, cu, ctx, H, Hk, D, D ** -0.5, n, scratch=sc) for q, kv in zip(qs, kvs)] * 3)
    return row(f"attn_prefill rows {n} heads {H}/{Hk}", us, 4 * out.numel(), 4.0 * visible_pairs(n, 0) * H * D)


def norms(cfg: ModelConfig, n: int) -> list[dict]:
    """The fused residual norm and the other row-wise kernels, beside the plain RMSNorm of the other families."""
    from . import ops as base
    from .engine.latent import PaddedSizes
    from .ops import latent as ops
    d, ff, m, dev = cfg.d_model, cfg.ff_width(0), cfg.mixers[0], "cuda"
    s = PaddedSizes.of(m)
    bf = dict(dtype=torch.bfloat16, device=dev)
    w = torch.ones(d, device=dev)
    k = min(copies_for(n * d * 12), 64)
    hs, ys, xs = [torch.randn(n, d, device=dev) for _ in range(k)], [torch.randn(n, d, **bf) for _ in range(k)], [torch.empty(n, d, **bf) for _ in range(k)]
    rows = [row(f"resid_norm rows {n} (two norms, residual update)", time_us([lambda h=h, y=y, x=x: ops.resid_norm(h, y, w, w_next=w, xn=x, eps=1e-6) for h, y, x in zip(hs, ys, xs)]), n * d * 12, 0),
            row(f"rmsnorm rows {n} (other families)", time_us([lambda h=h, x=x: base.rmsnorm(h, w, x, 1e-6) for h, x in zip(hs, xs)]), n * d * 6, 0)]
    k = min(copies_for(n * ff * 6), 64)
    gus, act = [torch.randn(n, 2 * ff, **bf) for _ in range(k)], torch.empty(n, ff, **bf)
    rows.append(row(f"gelu_mul rows {n}", time_us([lambda g=g: ops.gelu_mul(g, act) for g in gus]), n * ff * 6, 0))
    cols = m.q_rank + m.kv_rank + m.rot_dim
    bt, P, pages = page_tables(1, n, dev)
    k = min(copies_for(n * cols * 4), 64)
    downs, kv = [torch.randn(n, cols, **bf) for _ in range(k)], torch.zeros(pages, 64, s.width, **bf)
    cqs = [torch.empty(n, s.q_rank, **bf) for _ in range(k)]
    pos, sid = torch.arange(n, dtype=torch.int32, device=dev), torch.zeros(n, dtype=torch.int32, device=dev)
    ang, qn, kn = torch.rand(n, m.rotary.dims // 2, 2, device=dev), torch.ones(m.q_rank, device=dev), torch.ones(m.kv_rank, device=dev)
    rows.append(row(f"latent_prep rows {n}", time_us([lambda a=a, c=c: ops.latent_prep(a, qn, kn, ang, pos, sid, bt, c, kv, m.rot_dim, s.latent, 1e-6) for a, c in zip(downs, cqs)]), n * cols * 4, 0))
    return rows


def products(cfg: ModelConfig, rows_list=(1, 4, 8, 32)) -> list[dict]:
    """Matrix products of a decode step: bf16 weights here, 8-bit blocks on the quantised kernels for comparison."""
    from . import ops as base
    from .engine.dense import DenseLinear
    from .engine.latent import PaddedSizes
    from .gguf import GGMLType, quantize
    from .ops import latent as ops
    d, ff, m, dev = cfg.d_model, cfg.ff_width(0), cfg.mixers[0], "cuda"
    s = PaddedSizes.of(m)
    bf = dict(dtype=torch.bfloat16, device=dev)
    out = []
    shapes = {"down_a": (m.q_rank + m.kv_rank + m.rot_dim, d), "q_b": (s.heads * (s.dim + s.rot), s.q_rank), "wo": (d, s.heads * s.vdim), "down": (d, ff)}
    for rows in rows_list:
        for name, (n, k) in shapes.items():
            c = copies_for(n * k * 2)
            lins = [DenseLinear(torch.randn(n, k, **bf)) for _ in range(c)]
            x, y = torch.randn(rows, k, **bf), torch.empty(rows, n, **bf)
            kind = "gemv_dense" if rows <= ops.GEMV_MAX_ROWS else "cuBLAS"
            out.append(row(f"{name} [{n}, {k}] x {rows} rows ({kind})", time_us([lambda l=l: l(x, y) for l in lins]), n * k * 2, 2.0 * n * k * rows))
            del lins
        c = copies_for(ff * d * 4)
        lins = [DenseLinear(torch.randn(2 * ff, d, **bf)) for _ in range(c)]
        x, act, gu = torch.randn(rows, d, **bf), torch.empty(rows, ff, **bf), torch.empty(rows, 2 * ff, **bf)
        out.append(row(f"gate|up + gelu [{2 * ff}, {d}] x {rows} rows", time_us([lambda l=l: l.gelu(x, act, gu) for l in lins]), ff * d * 4, 4.0 * ff * d * rows))
        del lins
        if rows <= ops.GEMV_MAX_ROWS:
            c = copies_for(s.heads * s.dim * s.latent * 2)
            ws = [torch.randn(s.heads, s.latent, s.dim, **bf) for _ in range(c)]
            vs = [torch.randn(s.heads, s.vdim, s.latent, **bf) for _ in range(c)]
            q, ql, o = torch.randn(s.heads, rows, s.dim, **bf), torch.empty(s.heads, rows, s.latent, **bf), torch.empty(s.heads, rows, s.vdim, **bf)
            out.append(row(f"query into latent space x {rows} rows", time_us([lambda w=w: ops.gemv_dense(w, q, ql) for w in ws]), ws[0].numel() * 2, 0))
            out.append(row(f"values from latent space x {rows} rows", time_us([lambda w=w: ops.gemv_dense(w, ql, o) for w in vs]), vs[0].numel() * 2, 0))
        sc = base.scratch_for(torch.device("cuda", torch.cuda.current_device()))
        n, k = d, ff
        packs = [base.pack_matrix(quantize(torch.randn(n, k, device=dev) * 0.05, GGMLType.Q8_0), GGMLType.Q8_0, n, k)]
        for _ in range(copies_for(n * k) - 1):
            packs.append(replace(packs[0], data=packs[0].data.clone()))
        x, y = torch.randn(rows, k, **bf), torch.empty(rows, n, **bf)
        fn = (lambda w: base.gemv(w, x, y, scratch=sc)) if rows <= base.GEMV_MAX_ROWS else (lambda w: base.gemm(w, x, y, scratch=sc))
        out.append(row(f"down [{n}, {k}] x {rows} rows (other families: Q8_0 kernel)", time_us([lambda w=w: fn(w) for w in packs]), packs[0].data.numel(), 2.0 * n * k * rows))
    return out


def run(layers: int = 8, log=print) -> dict:
    big, gqa = SHAPES["pozivik-8b"], SHAPES["qwen3-8b"]
    kernels = []
    for batch, ctx in ((1, 4096), (8, 4096), (32, 2048), (128, 2048)):
        kernels += [latent_decode(big, batch, ctx), latent_decode(big, batch, ctx, False), gqa_decode(gqa, batch, min(ctx, big.mixers[0].window))]
    wide = big.with_(mixers=tuple(replace(m, window=4096) for m in big.mixers))
    kernels += [latent_decode(wide, 32, 4096), latent_decode(wide, 32, 4096, False), gqa_decode(gqa, 32, 4096)]
    for n in (1024, 4096):
        for window in (0, 1024):
            kernels += latent_prefill(big, n, window)[:2 if window else 4]
        kernels.append(gqa_prefill(gqa, n))
    for n in (32, 4096):
        kernels += norms(big, n)
    kernels += products(big)
    for k in kernels:
        log(json.dumps(k))
    models = []
    for batch, prompt in ((1, 2048), (32, 1024)):
        for cfg, recipe in ((cut(big, layers), "BF16"), (cut(gqa, layers), "BF16"), (cut(gqa, layers), "Q8_0")):
            models.append(whole_model(cfg, recipe, prompt, batch))
            log(json.dumps(models[-1]))
    return {"peaks": measured_peaks()[2], "l2": "inputs larger than L2", "kernels": kernels, "models": models}
