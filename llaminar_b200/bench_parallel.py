"""Throughput and kernel times of models with parallel layers, an average over depth, lightning attention and convolved attention (lagedra)
beside the like parts of the other families at equal size.

Used by `bench.py --parallel`.  Single kernels with their fraction of the memory or tensor roofline, and whole models (prefill and decode
tokens per second through the engine, random weights, a few layers of full size).  The like kernels: retention of zogepel-8b (a state of
the same size), grouped attention, residual norms and experts of kefasun-8b, experts of the sizes of qwen3-30b-a3b, attention of qwen3-8b.
"""
from __future__ import annotations

import json
from dataclasses import replace

import torch

from .bench_experts import _router, _scratch, grouped_decode, grouped_prefill
from .bench_experts import head_prep as like_prep
from .bench_experts import moe_sized
from .bench_latent import gqa_decode, gqa_prefill
from .bench_mixers import linear_decode, linear_prefill
from .bench_util import copies_for, cut, measured_peaks, page_tables, row, time_us, visible_pairs, whole_model
from .models.config import SHAPES, Experts, GroupedAttention, LightningAttention, ModelConfig, RopeScaling, Rotary, parallel_stack

BF, F32, I32 = ({"dtype": t, "device": "cuda"} for t in (torch.bfloat16, torch.float32, torch.int32))


def experts_sized(layers: int) -> ModelConfig:
    """The width, heads, experts and vocabulary of qwen3-30b-a3b with this family's layers."""
    q = SHAPES["qwen3-30b-a3b"]
    kinds = (LightningAttention(16, 128, 128, tuple(1.0 - 2.0 ** (-3.0 - i / 2) for i in range(16))),
             GroupedAttention(q.n_heads, q.n_kv_heads, 128, 128, 128 ** -0.5, Rotary(128, 2e5, RopeScaling(8.0, 4096, 32.0, 1.0)), 1024, softcap=30.0, qk_norm=False, conv=4, temperature=True, value_mix=True))
    e = Experts(q.n_experts, q.n_experts_used, q.expert_ff, 16, 8, 7.0, False)
    return parallel_stack("lagedra-30b-a3b", q.d_model, tuple(kinds[i % 2] for i in range(layers)), (e,) * layers, q.vocab_size, 32768)


# -- lightning attention ---------------------------------------------------------------------------------------------------------
def lightning_decode(m: LightningAttention, batch: int) -> list[dict]:
    """The recurrence (silu on what it reads), and norm and gate behind it."""
    from .ops import mixers as ops
    H, d, v = m.heads, m.dim, m.vdim
    nbytes = batch * 2 * H * d * v * 4
    k = copies_for(nbytes)
    rows, raw, out = torch.randn(batch, 2 * H * (d + v), **F32), torch.empty(batch, H * v, **F32), torch.empty(batch, H * v, **BF)
    states, decay, w = [torch.zeros(batch + 1, H, v, d, **F32) for _ in range(k)], torch.tensor(m.decay, **F32), torch.ones(H * v, **F32)
    pos, slots, offs = torch.full((batch,), 500, **I32), torch.arange(batch, **I32), [0, H * d, 2 * H * d, 2 * H * d + H * v]
    args = lambda s: (rows, offs, None, decay, None, 1.0, 1.0, None, pos, slots, (s,), v, None, False, raw, 1e-6)
    us = time_us([lambda s=s: ops.linear_rows(*args(s), silu_in=True, raw=True) for s in states])
    both = time_us([lambda s=s: (ops.linear_rows(*args(s), silu_in=True, raw=True), ops.joint_gate(raw, rows, offs[3], w, H * v, out, 1e-6)) for s in states])
    name, io = f"lightning batch {batch} heads {H} x {d} x {v}", 4 * rows.numel()
    return [row(f"linear_rows {name}", us, nbytes + io, 0), row(f"linear_rows + joint_gate {name}", both, nbytes + io, 0)]


def lightning_prefill(m: LightningAttention, n: int) -> list[dict]:
    """Prompts: silu in place, chunk sums, scan, outputs, norm and gate."""
    from .ops import dense
    from .ops import mixers as ops
    H, d, v, st = m.heads, m.dim, m.vdim, _scratch().status
    offs, cols = [0, H * d, 2 * H * d, 2 * H * d + H * v], 2 * H * (d + v)
    xs, states = [torch.randn(n, cols, **BF) for _ in range(3)], [torch.zeros(2, H, v, d, **F32) for _ in range(3)]
    decay, w, raw, out = torch.tensor(m.decay, **F32), torch.ones(H * v, **F32), torch.empty(n, H * v, **BF), torch.empty(n, H * v, **BF)
    cu, pos, slots, tables = torch.tensor([0, n], **I32), torch.arange(n, **I32), torch.zeros(1, **I32), ops.chunk_tables([0, n], "cuda")
    chunk = lambda i: ops.linear_chunk(xs[i], offs, None, decay, None, 1.0, 1.0, cu, pos, slots, (states[i],), v, None, False, out, 1e-6, tables, raw, st, only_raw=True)
    gate = lambda i: ops.joint_gate(raw, xs[i], offs[3], w, H * v, out, 1e-6)
    silu = lambda i: dense.activate(xs[i][:, :offs[3]], xs[i][:, :offs[3]], dense.ACT_SILU)
    flops, qkv = 2.0 * n * H * (64 * (d + v) + 2 * d * v), n * offs[3] * 2.0
    times = [time_us([lambda i=i: f(i) for i in range(3)] * 2) for f in (chunk, gate, silu)]
    all3 = time_us([lambda i=i: (silu(i), chunk(i), gate(i)) for i in range(3)] * 2)
    assert int(st[0]) == 0
    name = f"rows {n} heads {H} x {d} x {v}"
    return [row(f"linear_chunk lightning {name} (three launches)", times[0], qkv + n * H * v * 2.0, flops), row(f"joint_gate {name}", times[1], n * H * v * 6.0, 0),
            row(f"silu in place {name}", times[2], 2 * qkv, 0), row(f"silu + linear_chunk + joint_gate {name}", all3, 2.0 * n * H * (2 * d + 3 * v), flops)]


# -- convolved attention ---------------------------------------------------------------------------------------------------------
def conv_prep(m: GroupedAttention, n: int, decode: bool) -> dict:
    from .ops import grouped as ops
    H, G, D = m.heads, m.kv_heads, m.head_size
    cols, dt = (H + 2 * G) * D, F32 if decode else BF
    bt, P, pages = page_tables(n if decode else 1, 512 if decode else n, "cuda")
    seqs = n if decode else 1
    io = n * cols * (10 if decode else 4) + (n * cols * 4 * (m.conv - 1) if decode else 0)           # a decode step reads and writes the ring
    k = min(copies_for(io), 64)
    xs, qs = [torch.randn(n, cols, **dt) for _ in range(k)], [torch.empty(n, H, D, **BF) for _ in range(k)]
    kv, taps, rings = torch.zeros(pages, 2, G, 64, D, **BF), torch.randn(m.conv, cols, **F32), [torch.zeros(seqs + 1, m.conv, cols, **F32) for _ in range(k)]
    ang, gain, first, share = torch.rand(n, m.rotary.dims // 2, 2, device="cuda"), torch.ones(H, **F32), torch.zeros(n, G, D, **F32), torch.tensor([0.5], **F32)
    pos = torch.full((n,), 500, **I32) if decode else torch.arange(n, **I32)
    sid, slots, cu = torch.arange(n, **I32) if decode else torch.zeros(n, **I32), torch.arange(seqs, **I32), None if decode else torch.tensor([0, n], **I32)
    us = time_us([lambda x=x, q=q, r=r: ops.conv_prep(x, taps, r, slots, cu, ang, gain, first, share, pos, sid, bt, q, kv) for x, q, r in zip(xs, qs, rings)])
    return row(f"conv_prep {'batch' if decode else 'rows'} {n} heads {H}/{G} taps {m.conv}, values mixed", us, io + n * G * D * 4, 0)


def window_attention(m: GroupedAttention, batch: int, ctx: int, n: int) -> list[dict]:
    """Windowed, soft-capped attention: a decode step over a long context, and a prompt."""
    from .ops import grouped as ops
    H, G, D, sc = m.heads, m.kv_heads, m.head_size, _scratch()
    bt, P, pages = page_tables(batch, ctx, "cuda")
    keys = min(ctx, m.window)
    nbytes = batch * keys * 2 * G * D * 2
    kvs = [torch.randn(pages, 2, G, 64, D, **BF) for _ in range(copies_for(nbytes))]
    q, o, lens = torch.randn(batch, H, D, **BF), torch.empty(batch, H * D, **BF), torch.full((batch,), ctx, **I32)
    sp = ops.decode_splits(batch, G, D, P, m.window, sc)
    us = time_us([lambda kv=kv: ops.attn_decode(q, kv, o, bt, lens, m.scale, sp, m.window, None, None, sc, softcap=m.softcap) for kv in kvs])
    out = [row(f"attn_decode window {m.window} softcap batch {batch} context {ctx} heads {H}/{G}", us, nbytes + 4 * q.numel(), 4.0 * batch * H * keys * D)]
    del kvs
    bt, P, pages = page_tables(1, n, "cuda")
    qs, kvs, o = [torch.randn(n, H, D, **BF) for _ in range(3)], [torch.randn(pages, 2, G, 64, D, **BF) for _ in range(3)], torch.empty(n, H * D, **BF)
    cu, start, st = torch.tensor([0, n], **I32), torch.zeros(1, **I32), sc.status if ops.prefill_tc(D, n) else None
    us = time_us([lambda q=q, kv=kv: ops.attn_prefill(q, kv, o, bt, cu, start, m.scale, n, m.window, None, None, st, softcap=m.softcap) for q, kv in zip(qs, kvs)] * 3)
    out.append(row(f"attn_prefill window {m.window} softcap rows {n} heads {H}/{G}", us, 4 * o.numel() + 4 * n * G * D, 4.0 * visible_pairs(n, m.window) * H * D))
    return out


# -- rows ------------------------------------------------------------------------------------------------------------------------
def row_wise(d: int, ff: int, e: Experts, n: int) -> list[dict]:
    from .ops import dense as ops
    g, w1, out = torch.ones(1, **F32), torch.ones(d, **F32), []
    x0, x1 = torch.empty(n, d, **BF), torch.empty(n, d, **BF)
    for past in (1, 4, 8, 16):
        k = min(copies_for(n * d * (16 + 4 * past)), 32)
        streams, hs = [torch.randn(past + 1, n, d, **F32) for _ in range(k)], [torch.randn(n, d, **F32) for _ in range(k)]
        y, z, w = torch.randn(n, d, **BF), torch.randn(n, d, **BF), torch.rand(past + 1, **F32)
        us = time_us([lambda i=i: ops.depth_mix(hs[i], y, z, past=streams[i], n_past=past, w=w, norms=((g, x0), (g, x1)), eps=1e-6) for i in range(k)])
        out.append(row(f"depth_mix rows {n} of {d}, {past} streams, two norms", us, n * d * (2 * 2 + 8 + 4 + 4 * past + 2 * 2), 0))
        if past == 4:
            parts, wt, at = torch.randn(n * e.top, d, **BF), torch.rand(n, e.top, **F32), torch.randperm(n * e.top, device="cuda").int()
            us = time_us([lambda i=i: ops.depth_mix(hs[i], y, parts, z_rows=at if n > 64 else None, z_w=wt, past=streams[i], n_past=past, w=w, norms=((g, x0), (g, x1)), eps=1e-6) for i in range(k)])
            out.append(row(f"depth_mix rows {n} of {d}, {past} streams, two norms, sum of {e.top} experts", us, n * d * (2 + 2 * e.top + 8 + 4 + 4 * past + 2 * 2), 0))
            k = min(copies_for(n * d * 12), 64)
            hs, ys, xs = [torch.randn(n, d, **F32) for _ in range(k)], [torch.randn(n * e.top, d, **BF) for _ in range(min(k, 8))], [torch.empty(n, d, **BF) for _ in range(k)]
            us = time_us([lambda i=i: ops.resid_norm(hs[i], ys[i % len(ys)], w1, w_next=w1, xn=xs[i], eps=1e-6, y_rows=at if n > 64 else None, y_w=wt) for i in range(k)])
            out.append(row(f"resid_norm rows {n} of {d}, sum of {e.top} experts (kefasun)", us, n * d * (10 + 2 * e.top), 0))
            us = time_us([lambda i=i: ops.resid_norm(hs[i], ys[i % len(ys)][:n], w1, w_next=w1, xn=xs[i], eps=1e-6) for i in range(k)])
            out.append(row(f"resid_norm rows {n} of {d} (kefasun)", us, n * d * 12, 0))
        del streams
    k = min(copies_for(n * ff * 4), 32)
    gu, act = [torch.randn(n, 2 * ff, **BF) for _ in range(k)], torch.empty(n, ff, **BF)
    out.append(row(f"activate gelu rows {n} of {ff}", time_us([lambda u=u: ops.activate(u.view(2 * n, ff)[:n], act, ops.ACT_GELU) for u in gu]), n * ff * 4, 0))
    out.append(row(f"activate gelu pairs rows {n} of {ff} (pozivik)", time_us([lambda u=u: ops.activate(u, act, ops.ACT_GELU_MUL) for u in gu]), n * ff * 6, 0))
    return out


def up_product(d: int, ff: int, rows: int) -> list[dict]:
    from .engine.dense import DenseLinear
    from .ops import dense as ops
    c, out = copies_for(ff * d * 2), []
    x, act, raw = torch.randn(rows, d, **BF), torch.empty(rows, ff, **BF), torch.empty(rows, 2 * ff, **BF)
    for name, kind, n in (("up + gelu", ops.ACT_GELU, ff), ("gate|up + gelu (pozivik)", ops.ACT_GELU_MUL, 2 * ff)):
        lins = [DenseLinear(torch.randn(n, d, **BF)) for _ in range(c)]
        out.append(row(f"{name} [{n}, {d}] x {rows} rows", time_us([lambda l=l: l.activated(x, act, raw.view(-1)[:rows * n].view(rows, n), kind) for l in lins]), n * d * 2, 2.0 * n * d * rows))
        del lins
    return out


# -- experts: with groups and limits, and without --------------------------------------------------------------------------------
def experts(d: int, e: Experts, T: int) -> list[dict]:
    from .ops import experts as ops
    P, new, status, out = T * e.top, torch.empty, _scratch().status, []
    x, router, bias = _router(T, d, e)
    ids, wt, ranks, place, counts = new(T, e.top, **I32), new(T, e.top, **F32), new(P, **I32), new(P, **I32), torch.zeros(e.n, **I32)
    act, y, xs, few = new(P, e.ff, **BF), new(P, d, **BF), new(P, d, **BF), P <= 512
    logits = torch.mm(x, router.t(), out_dtype=torch.float32)
    for name, groups, keep, b in ((f"{e.keep} of {e.groups} groups", e.groups, e.keep, None), ("(kefasun)", 1, 1, bias)):
        if few:
            routers = [router.clone() for _ in range(copies_for(router.numel() * 2))]
            us = time_us([lambda r=r: ops.expert_route(b, ids, wt, x=x, router=r, groups=groups, keep=keep) for r in routers])
            out.append(row(f"expert_route {T} tokens, {e.n} experts of which {e.top}, {name}", us, router.numel() * 2 + 2 * x.numel(), 0))
        else:
            us = time_us([lambda: (counts.zero_(), ops.expert_route(b, ids, wt, logits=logits, counts=counts, ranks=ranks, groups=groups, keep=keep))] * 20)
            out.append(row(f"expert_route {T} tokens, {e.n} experts of which {e.top}, logits given, {name}", us, 4 * logits.numel() + 8 * P, 0))
    counts.zero_()
    ops.expert_route(None, ids, wt, logits=logits, counts=counts, ranks=ranks, groups=e.groups, keep=e.keep)
    used = int((counts > 0).sum())
    ws = [torch.randn(e.n, 2 * e.ff, d, **BF) for _ in range(3)]
    turns = max(1, min(8, copies_for(used * 2 * e.ff * d * 2) // 3))
    shifts = [((ids + s * (e.n // turns)) % e.n).contiguous() for s in range(turns)]
    if not few:
        ops.expert_place(x, ids, ranks, counts, place, xs)
    for name, limit in (("limited pairs", 7.0), ("silu pairs (kefasun)", 0.0)):
        if few:
            us = time_us([lambda w=w, i=i: ops.expert_rows(w, x, i, act, e.top, True, limit) for i in shifts for w in ws])
            out.append(row(f"expert_rows gate|up {name} [{e.n}, {2 * e.ff}, {d}] {T} tokens x {e.top}, {used} experts used", us, used * 4.0 * e.ff * d, 4.0 * P * e.ff * d))
        else:
            us = time_us([lambda w=w: ops.expert_grouped(w, xs, counts, act, True, status, limit) for w in ws * 2])
            out.append(row(f"expert_grouped gate|up {name} [{e.n}, {2 * e.ff}, {d}] {P} rows", us, 2 * (used * 2.0 * e.ff * d + P * (d + e.ff)), 4.0 * P * e.ff * d))
    assert int(status[0]) == 0
    return out


def run(layers: int = 8, log=print) -> dict:
    big, kef, zog, gqa, moe = (SHAPES[n] for n in ("lagedra-8b", "kefasun-8b", "zogepel-8b", "qwen3-8b", "qwen3-30b-a3b"))
    kernels = []

    def add(*rows):
        for r in rows:
            kernels.append(r)
            log(json.dumps(r))
        torch.cuda.empty_cache()
    light, attn, capped, ret = big.mixers[0], big.mixers[1], kef.mixers[2], zog.mixers[1].right
    for batch in (1, 8, 32):
        add(*lightning_decode(light, batch), linear_decode(ret, batch))
    for n in (1024, 4096):
        add(*lightning_prefill(light, n), linear_prefill(ret, n))
    for n in (1, 32):
        add(conv_prep(attn, n, True), *like_prep(capped, n))
    for n in (1024, 4096):
        add(conv_prep(attn, n, False), *like_prep(capped, n))
    for batch, n in ((1, 1024), (32, 4096)):
        add(*window_attention(attn, batch, 2048, n), grouped_decode(replace(capped, gate="head"), batch, 1024), gqa_decode(gqa, batch, 1024), grouped_prefill(capped, n), gqa_prefill(gqa, n))
    wide = big.experts_of(1)
    for n in (1, 32, 4096):
        add(*row_wise(big.d_model, big.d_ff, wide, n))
    for n in (1, 8, 32):
        add(*up_product(big.d_model, big.d_ff, n))
    narrow = experts_sized(1).experts_of(0)
    for T in (1, 32, 4096):
        add(*experts(moe.d_model, narrow, T), *experts(big.d_model, wide, T))
    models = []
    for batch, prompt in ((1, 2048), (32, 1024)):
        for c in (cut(big, layers), cut(kef, layers), cut(zog, layers), cut(gqa, layers), experts_sized(layers), moe_sized(layers)):
            models.append(whole_model(c, "BF16", prompt, batch))
            log(json.dumps(models[-1]))
    return {"peaks": measured_peaks()[2], "l2": "inputs larger than L2", "kernels": kernels, "models": models}
