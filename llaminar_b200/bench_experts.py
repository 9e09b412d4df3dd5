"""Throughput and kernel times of models with routed experts and gated grouped attention (kefasun) beside the like parts of the other
families at equal size.

Used by `bench.py --experts`.  Single kernels with their fraction of the memory or tensor roofline, and whole models (prefill and decode
tokens per second through the engine, random weights, a few layers of full size).  The like kernels: the experts of qwen3-30b-a3b (same
sizes, 3-bit codebook weights), grouped-query attention of qwen3-8b, latent attention, norms and activations of pozivik-8b.
"""
from __future__ import annotations

import json
from dataclasses import replace

import torch

from .bench_latent import gqa_decode, gqa_prefill
from .bench_util import copies_for, cut, measured_peaks, page_tables, row, time_us, visible_pairs, whole_model
from .models.config import SHAPES, Experts, GroupedAttention, LatentAttention, ModelConfig, Rotary, attention_stack

BF, F32, I32 = ({"dtype": t, "device": "cuda"} for t in (torch.bfloat16, torch.float32, torch.int32))


def _scratch():
    from . import ops
    return ops.scratch_for(torch.device("cuda", torch.cuda.current_device()))


def moe_sized(layers: int) -> ModelConfig:
    """The layers of qwen3-30b-a3b (width, heads, experts, vocabulary) with this family's attention."""
    q = SHAPES["qwen3-30b-a3b"]
    kinds = (GroupedAttention(q.n_heads, q.n_kv_heads, 128, 128, 128 ** -0.5, Rotary(64, 2e5, interleaved=True), chunk=4096, null_key=True, gate="head"),
             GroupedAttention(q.n_heads, q.n_kv_heads, 128, 128, 128 ** -0.5, Rotary(128, 8e5), softcap=40.0, gate="value"))
    mixers = tuple(kinds[i % 2] for i in range(layers))
    return attention_stack("kefasun-30b-a3b", q.d_model, mixers, (Experts(q.n_experts, q.n_experts_used, q.expert_ff),) * layers, q.vocab_size)


# -- experts ---------------------------------------------------------------------------------------------------------------------
def _router(T: int, d: int, e: Experts):
    g = torch.Generator(device="cuda").manual_seed(1)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    return rnd(T, d).bfloat16(), (rnd(e.n, d) * 2 * d ** -0.5).bfloat16(), torch.zeros(e.n, device="cuda")


def experts_few(d: int, e: Experts, T: int) -> list[dict]:
    """A decode step: route, gate|up with silu, down.  Bytes: the matrices of the experts that are chosen."""
    from .ops import experts as ops
    P, new = T * e.top, torch.empty
    x, router, bias = _router(T, d, e)
    ids, wt = new(T, e.top, **I32), new(T, e.top, **F32)
    routers = [router.clone() for _ in range(copies_for(router.numel() * 2))]
    out = [row(f"expert_route {T} tokens, {e.n} experts of which {e.top}, width {d}",
               time_us([lambda r=r: ops.expert_route(bias, ids, wt, x=x, router=r) for r in routers]), router.numel() * 2 + 2 * x.numel(), 0)]
    used = int(ids.unique().numel())
    act, y = new(P, e.ff, **BF), new(P, d, **BF)
    for name, n, k, pair in (("gate|up + silu", 2 * e.ff, d, True), ("down", d, e.ff, False)):
        nbytes = used * n * k * 2
        ws = [torch.randn(e.n, n, k, **BF) for _ in range(3 if e.n * n * k > 1 << 27 else 6)]
        # few experts in use: every copy lets other ones be chosen, so that the weights come from memory
        turns = max(1, min(16, copies_for(nbytes) // len(ws)))
        shifts = [((ids + s * (e.n // turns)) % e.n).contiguous() for s in range(turns)]
        calls = [lambda w=w, i=i: (ops.expert_rows(w, x, i, act, e.top, True) if pair else ops.expert_rows(w, act, i, y, 1, False)) for i in shifts for w in ws]
        out.append(row(f"expert_rows {name} [{e.n}, {n}, {k}] {T} tokens x {e.top}, {used} experts used", time_us(calls), nbytes, 2.0 * P * n * k))
        del ws, calls
    return out


def experts_many(d: int, e: Experts, T: int) -> list[dict]:
    """Prompts: choice, sort and copy, both grouped products."""
    from .ops import experts as ops
    P, new, status = T * e.top, torch.empty, _scratch().status
    x, router, bias = _router(T, d, e)
    ids, wt, ranks, place, counts = new(T, e.top, **I32), new(T, e.top, **F32), new(P, **I32), new(P, **I32), torch.zeros(e.n, **I32)
    xs, act, y = new(P, d, **BF), new(P, e.ff, **BF), new(P, d, **BF)

    def choose():
        counts.zero_()
        ops.expert_route(bias, ids, wt, logits=torch.mm(x, router.t(), out_dtype=torch.float32), counts=counts, ranks=ranks)
    out = [row(f"router product + expert_route {T} tokens, {e.n} experts of which {e.top}", time_us([choose] * 20), 2 * x.numel() + 4 * T * e.n, 2.0 * T * e.n * d)]
    choose()
    out.append(row(f"expert_place {P} rows of {d}", time_us([lambda: ops.expert_place(x, ids, ranks, counts, place, xs)] * 20), 2 * (x.numel() + xs.numel()), 0))
    used = int((counts > 0).sum())
    for name, n, k, pair in (("gate|up + silu", 2 * e.ff, d, True), ("down", d, e.ff, False)):
        ws = [torch.randn(e.n, n, k, **BF) for _ in range(3)]
        calls = [lambda w=w: (ops.expert_grouped(w, xs, counts, act, True, status) if pair else ops.expert_grouped(w, act, counts, y, False, status)) for w in ws]
        nbytes = 2 * (used * n * k + P * (k + (n // 2 if pair else n)))
        out.append(row(f"expert_grouped {name} [{e.n}, {n}, {k}] {P} rows", time_us(calls * 2), nbytes, 2.0 * P * n * k))
        del ws, calls
    assert int(status[0]) == 0
    return out


def quantised_experts(d: int, e: Experts, T: int) -> list[dict]:
    """The same layer on the quantised kernels (IQ3_S): few rows as three launches, prompts as two grouped products."""
    from . import ops
    from .gguf.constants import BLOCK_GEOMETRY, GGMLType
    from .ops.layout import pack_experts
    q3, E, k, sc, zi = GGMLType.IQ3_S, e.n, e.top, _scratch(), torch.zeros
    el, by = BLOCK_GEOMETRY[q3]

    def slab(n, kk):
        raw = torch.randint(0, 256, (E * n * kk // el * by,), dtype=torch.uint8, device="cuda")
        raw.view(torch.int16).bitwise_and_(0x1FFF)
        return pack_experts(raw, q3, E, n, kk), raw.numel() / E
    (gu, b1), (dn, b2) = slab(2 * e.ff, d), slab(d, e.ff)
    copy = lambda p: [p] + [replace(p, data=p.data.clone()) for _ in range(3)]
    h, w = torch.randn(T, d, **F32), torch.ones(d, device="cuda")
    _, router, _ = _router(T, d, e)
    P, ids, wt = T * k, zi(T, k, **I32), zi(T, k, **F32)
    act, y = zi(P, e.ff, **BF), zi(P, d, **F32)
    if P > 512:
        xn = zi(T, d, **BF)
        ops.moe_route_only(h, w, 1e-6, router, k, True, ids, wt, xn)
        order = torch.argsort(ids.view(-1).long(), stable=True)
        counts, avg = torch.bincount(ids.view(-1).long(), minlength=E).int(), P // E
        bm = 256 if avg >= 192 else (128 if avg >= 96 else 64)
        off = lambda c: torch.cat([zi(1, **I32), torch.cumsum(c, 0, dtype=torch.int32)])
        ro, to, xg = off(counts), off((counts + bm - 1) // bm), xn.index_select(0, order // k)
        a = time_us([lambda p=p: ops.gemm_grouped(p, xg, act, ro, to, bm, epi=ops.EPI_SWIGLU, scratch=sc) for p in copy(gu)])
        b = time_us([lambda p=p: ops.gemm_grouped(p, act, y, ro, to, bm, scratch=sc) for p in copy(dn)])
        return [row(f"gemm_grouped gate|up + silu [{E}, {2 * e.ff}, {d}] {P} rows (quantised experts)", a, b1 * E + 2 * P * (d + e.ff), 4.0 * P * e.ff * d),
                row(f"gemm_grouped down [{E}, {d}, {e.ff}] {P} rows (quantised experts)", b, b2 * E + P * (2 * e.ff + 4 * d), 2.0 * P * e.ff * d)]
    z = E + (P + 3) // 4
    items, n_items, ticket, tt, ys = zi(z * ops.MOE_ITEM_INTS, **I32), zi(1, **I32), zi(1, **I32), zi(d // 128, **I32), zi(P, d, **F32)
    route = time_us([lambda: ops.moe_route(h, w, 1e-6, router, k, True, 0, E, ids, wt, items, n_items, ticket)] * 20)
    used = int(ids.unique().numel())
    a = time_us([lambda p=p: ops.moe_gate_up(p, h, w, 1e-6, act, items, n_items, k, z, scratch=sc) for p in copy(gu)])
    b = time_us([lambda p=p: ops.moe_down_combine(p, act, ys, items, n_items, z, ids, wt, k, 0, E, h, tt, scratch=sc) for p in copy(dn)])
    return [row(f"moe_route {T} tokens, {E} experts (with norm and work list, quantised experts)", route, router.numel() * 2 + 4 * h.numel(), 0),
            row(f"moe_gate_up [{E}, {2 * e.ff}, {d}] {T} tokens x {k} (quantised experts)", a, b1 * used, 4.0 * P * e.ff * d),
            row(f"moe_down_combine [{E}, {d}, {e.ff}] {T} tokens x {k} (quantised experts)", b, b2 * used, 2.0 * P * e.ff * d)]


# -- attention -------------------------------------------------------------------------------------------------------------------
def _describe(m: GroupedAttention) -> str:
    return f"{'chunk ' + str(m.chunk) + ' ' if m.chunk else ''}{'softcap ' if m.softcap else ''}{m.gate} gate heads {m.heads}/{m.kv_heads}"


def grouped_decode(m: GroupedAttention, batch: int, keys: int) -> dict:
    from .ops import grouped as ops
    H, G, D, sc = m.heads, m.kv_heads, m.head_size, _scratch()
    bt, P, pages = page_tables(batch, keys, "cuda")
    nbytes = batch * keys * 2 * G * D * 2
    kvs = [torch.randn(pages, 2, G, 64, D, **BF) for _ in range(copies_for(nbytes))]
    q, o, gate = torch.randn(batch, H, D, **BF), torch.empty(batch, H * D, **BF), torch.randn(batch, m.gate_width, **F32)
    sink, lens = torch.zeros(H, **F32) if m.null_key else None, torch.full((batch,), keys, **I32)
    sp = ops.decode_splits(batch, G, D, P, 0, sc, m.chunk)
    us = time_us([lambda kv=kv: ops.attn_decode(q, kv, o, bt, lens, m.scale, sp, 0, sink, gate, sc, chunk=m.chunk, softcap=m.softcap) for kv in kvs])
    return row(f"attn_decode {_describe(m)} batch {batch} keys {keys}", us, nbytes + 4 * q.numel() + 4 * gate.numel(), 4.0 * batch * H * keys * D)


def grouped_prefill(m: GroupedAttention, n: int) -> dict:
    from .ops import grouped as ops
    H, G, D, sc = m.heads, m.kv_heads, m.head_size, _scratch()
    bt, P, pages = page_tables(1, n, "cuda")
    qs, kvs = [torch.randn(n, H, D, **BF) for _ in range(3)], [torch.randn(pages, 2, G, 64, D, **BF) for _ in range(3)]
    out, gate, sink = torch.empty(n, H * D, **BF), torch.randn(n, m.gate_width, **BF), torch.zeros(H, **F32) if m.null_key else None
    cu, ctx = torch.tensor([0, n], **I32), torch.zeros(1, **I32)
    st = sc.status if ops.prefill_tc(D, n) else None
    us = time_us([lambda q=q, kv=kv: ops.attn_prefill(q, kv, out, bt, cu, ctx, m.scale, n, 0, sink, gate, st, chunk=m.chunk, softcap=m.softcap) for q, kv in zip(qs, kvs)] * 3)
    pairs = visible_pairs(n, 0) if not m.chunk else sum(visible_pairs(min(m.chunk, n - i), 0) for i in range(0, n, m.chunk))
    return row(f"attn_prefill {_describe(m)} rows {n}", us, 4 * out.numel() + 2 * gate.numel(), 4.0 * pairs * H * D)


def head_prep(m: GroupedAttention, n: int) -> list[dict]:
    from . import ops as base
    from .ops import grouped as ops
    H, G, D = m.heads, m.kv_heads, m.head_size
    cols = (H + 2 * G) * D
    bt, P, pages = page_tables(1, n, "cuda")
    k = min(copies_for(n * cols * 4), 64)
    dt = F32 if n <= 64 else BF
    xs, qs = [torch.randn(n, cols, **dt) for _ in range(k)], [torch.empty(n, H, D, **BF) for _ in range(k)]
    kv, w, ang = torch.zeros(pages, 2, G, 64, D, **BF), torch.ones(D, **F32), torch.rand(n, m.rotary.dims // 2, 2, device="cuda")
    pos, sid = torch.arange(n, **I32), torch.zeros(n, **I32)
    ours = time_us([lambda x=x, q=q: ops.head_prep(x, 0, H * D, (H + G) * D, w, w, ang, pos, sid, bt, q, kv, D, 1e-6) for x, q in zip(xs, qs)])
    xs = [x.bfloat16() for x in xs]
    theirs = time_us([lambda x=x, q=q: base.rope_kv(x, q, kv, w, w, pos, sid, bt, H, G, D, 1e6, 1e-6) for x, q in zip(xs, qs)])
    return [row(f"head_prep rows {n} heads {H}/{G}", ours, n * cols * (6 if n <= 64 else 4), 0), row(f"rope_kv rows {n} heads {H}/{G} (qwen3-8b)", theirs, n * cols * 4, 0)]


def latent_gates(m: LatentAttention, n: int) -> list[dict]:
    """Prompt attention with the gate in the epilogue and without."""
    from .engine.latent import PaddedSizes
    from .ops import latent as ops
    s, st, out = PaddedSizes.of(m), _scratch().status, []
    q, k = [torch.randn(n, s.heads, s.dim + s.rot, **BF) for _ in range(3)], [torch.randn(n, s.heads * s.dim, **BF) for _ in range(3)]
    v = [torch.randn(s.heads * s.vdim, n, **BF) for _ in range(3)]
    lat, o = torch.randn(n, s.width, **BF), torch.empty(n, s.heads * s.vdim, **BF)
    ang, sink, gate = torch.rand(n, m.rotary.dims // 2, 2, device="cuda"), torch.zeros(s.heads, **F32), torch.randn(n, s.heads * s.vdim, **BF)
    seqs = torch.tensor([[0, 0, n, 0, 0, 0, n, 0]], **I32)
    pairs = visible_pairs(n, m.window)
    for name, g in (("with gate", gate), ("(pozivik)", None)):
        us = time_us([lambda i=i: ops.latent_chunk(q[i], ang, k[i], v[i], lat, s.latent, seqs, n, o, s.dim, s.rot, s.vdim, m.window, m.scale, sink, st, g) for i in range(3)] * 3)
        out.append(row(f"latent_chunk {name} rows {n} window {m.window} heads {s.heads}", us, 2 * (q[0].numel() + 2 * k[0].numel() + o.numel() * (2 if g is not None else 1)),
                       2.0 * pairs * s.heads * (m.dim + m.rot_dim + m.vdim)))
    return out


def latent_gates_decode(m: LatentAttention, rows: int) -> list[dict]:
    """What gates the values of a decode step: the product that brings them out of the latent space, or a kernel behind it."""
    from .engine.latent import PaddedSizes
    from .ops import latent as ops
    s, out = PaddedSizes.of(m), []
    gate, o = torch.randn(rows, s.heads * s.vdim, **BF), torch.empty(rows, s.heads, s.vdim, **BF)
    side = (gate, 0, s.heads * s.vdim, None)
    if rows <= ops.GEMV_MAX_ROWS:
        vs, ql = [torch.randn(s.heads, s.vdim, s.latent, **BF) for _ in range(copies_for(s.heads * s.vdim * s.latent * 2))], torch.randn(s.heads, rows, s.latent, **BF)
        for name, kw in (("with gate", dict(act=ops.ACT_GATE, side=side)), ("(pozivik)", {})):
            out.append(row(f"values from latent space {name} x {rows} rows", time_us([lambda v=v: ops.gemv_dense(v, ql, o.transpose(0, 1), **kw) for v in vs]), vs[0].numel() * 2, 0))
    else:
        flat = o.view(rows, -1)
        out.append(row(f"gate x {rows} rows of {s.heads * s.vdim}", time_us([lambda: ops.activate(flat, flat, ops.ACT_GATE, side)] * 20), 6 * flat.numel(), 0))
    return out


# -- rows ------------------------------------------------------------------------------------------------------------------------
def row_wise(d: int, ff: int, e: Experts, n: int) -> list[dict]:
    from .ops import dense as ops
    w, k, out = torch.ones(d, **F32), min(copies_for(n * d * 12), 64), []
    hs, ys, xs = [torch.randn(n, d, **F32) for _ in range(k)], [torch.randn(n * e.top, d, **BF) for _ in range(min(k, 8))], [torch.empty(n, d, **BF) for _ in range(k)]
    wt, at = torch.rand(n, e.top, **F32), torch.randperm(n * e.top, device="cuda").int()
    us = time_us([lambda i=i: ops.resid_norm(hs[i], ys[i % len(ys)], w, w_next=w, xn=xs[i], eps=1e-6, y_rows=at if n > 64 else None, y_w=wt) for i in range(k)])
    out.append(row(f"resid_norm rows {n} of {d}, sum of {e.top} experts", us, n * d * (10 + 2 * e.top), 0))
    us = time_us([lambda i=i: ops.resid_norm(hs[i], ys[i % len(ys)][:n], w, w_next=w, xn=xs[i], eps=1e-6) for i in range(k)])
    out.append(row(f"resid_norm rows {n} of {d} (pozivik)", us, n * d * 12, 0))
    del ys
    k = min(copies_for(n * ff * 6), 32)
    gu, act = [torch.randn(n, 2 * ff, **BF) for _ in range(k)], torch.empty(n, ff, **BF)
    for name, kind in (("silu pairs", ops.ACT_SILU_MUL), ("gelu pairs (pozivik)", ops.ACT_GELU_MUL)):
        out.append(row(f"activate {name} rows {n} of {ff}", time_us([lambda g=g: ops.activate(g, act, kind) for g in gu]), n * ff * 6, 0))
    return out


def run(layers: int = 8, log=print) -> dict:
    big, lat, gqa, moe = SHAPES["kefasun-8b"], SHAPES["pozivik-8b"], SHAPES["qwen3-8b"], SHAPES["qwen3-30b-a3b"]
    kernels = []

    def add(*rows):
        for r in rows:
            kernels.append(r)
            log(json.dumps(r))
        torch.cuda.empty_cache()
    d, e, wide = moe.d_model, Experts(moe.n_experts, moe.n_experts_used, moe.expert_ff), big.experts_of(1)
    for T in (1, 8, 32, 64):
        add(*experts_few(d, e, T), *quantised_experts(d, e, T))
    for T in (1024, 4096):
        add(*experts_many(d, e, T), *quantised_experts(d, e, T))
    for T in (1, 32):
        add(*experts_few(big.d_model, wide, T))
    add(*experts_many(big.d_model, wide, 4096))
    chunked, latent, capped = big.mixers[:3]
    for batch, keys in ((1, 1024), (8, 1024), (32, 1024), (32, 4096)):
        add(grouped_decode(replace(chunked, chunk=keys), batch, keys), grouped_decode(capped, batch, keys), gqa_decode(gqa, batch, keys))
    for n in (1024, 4096):
        add(grouped_prefill(chunked, n), grouped_prefill(replace(chunked, chunk=0), n), grouped_prefill(capped, n), gqa_prefill(gqa, n), *latent_gates(latent, n))
    for rows in (1, 8, 32):
        add(*latent_gates_decode(latent, rows))
    for n in (32, 4096):
        add(*head_prep(capped, n), *row_wise(big.d_model, big.d_ff, wide, n))
    models = []
    for batch, prompt in ((1, 2048), (32, 1024)):
        for c in (cut(big, layers), cut(lat, layers), cut(gqa, layers), moe_sized(layers), cut(moe, layers)):
            models.append(whole_model(c, "Q4_K_M" if c.is_moe else "BF16", prompt, batch))
            log(json.dumps(models[-1]))
    return {"peaks": measured_peaks()[2], "l2": "inputs larger than L2", "kernels": kernels, "models": models}
