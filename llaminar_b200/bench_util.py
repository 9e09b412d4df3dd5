"""What the kernel and model benchmarks share: timing of captured launches, roofline fractions, throughput of whole models.

Kernels are timed with CUDA events around a captured graph of many launches that walk over buffers larger than L2 together.
"""
from __future__ import annotations

import json
import os
import statistics

import torch

from .models.config import ModelConfig

L2_BYTES = 126 << 20


def measured_peaks() -> tuple[float, float, str]:
    """(memory bandwidth in bytes/s, bf16 FLOP/s, where they come from)"""
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        p = json.load(open(path))
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def copies_for(nbytes: int) -> int:
    """How many copies of a kernel's data make its working set larger than L2."""
    return max(2, min(256, -(-2 * L2_BYTES // max(nbytes, 1))))


def time_us(calls: list, reps: int = 5) -> float:
    """Device time of one call: `calls` (closures over different buffers) captured back to back in a graph, median of replays."""
    s = torch.cuda.Stream()
    s.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(s):
        for c in calls[:3]:
            c()
    torch.cuda.current_stream().wait_stream(s)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for c in calls:
            c()
    for _ in range(3):
        g.replay()
    out = []
    for _ in range(reps):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        g.replay()
        b.record()
        torch.cuda.synchronize()
        out.append(a.elapsed_time(b) * 1e3 / len(calls))
    return statistics.median(out)


def row(name: str, us: float, nbytes: float, flops: float) -> dict:
    bw, tf, _ = measured_peaks()
    roof = max(nbytes / bw, flops / tf) * 1e6
    return {"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "fraction": round(roof / us, 3),
            "bound": "memory" if nbytes / bw >= flops / tf else "tensor"}


def visible_pairs(n: int, window: int) -> int:
    """Query-key pairs of a causal prompt of n tokens."""
    return sum(min(i + 1, window) if window else i + 1 for i in range(n))


def page_tables(batch: int, ctx: int, dev):
    P = -(-ctx // 64)
    bt = (torch.randperm(batch * P, device=dev).to(torch.int32) + 1).view(batch, P).contiguous()
    return bt, P, batch * P + 1


def whole_model(cfg: ModelConfig, recipe: str, prompt: int, batch: int, steps: int = 32) -> dict:
    """Prefill and decode tokens per second through the engine, device-timed."""
    from .engine.engine import LLMEngine
    from .engine.sampling import SamplingParams
    from .models.synth import synthesize
    w = synthesize(cfg, recipe, seed=0, device="cuda", with_tokenizer=False)
    eng = LLMEngine(w, device="cuda", max_batch=batch, max_context=prompt + 2 * steps + 80, max_prefill_tokens=8192)
    del w
    g = torch.Generator().manual_seed(1)
    sp = SamplingParams(temperature=0.0, max_tokens=10 ** 6, ignore_eos=True)
    make = lambda: [torch.randint(0, cfg.vocab_size, (prompt,), generator=g).tolist() for _ in range(batch)]
    for warm in (True, False):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        reqs = [eng.add_request(p, sp) for p in make()]
        torch.cuda.synchronize()
        a.record()
        while eng.waiting:
            eng.step()
        b.record()
        torch.cuda.synchronize()
        pre = batch * prompt / (a.elapsed_time(b) / 1e3)
        if warm:
            for r in reqs:
                eng.abort(r.rid)
    for _ in range(4):
        eng.step()
    evs = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(steps)]
    eng.step_events = list(evs)
    for _ in range(steps):
        eng.step()
    torch.cuda.synchronize()
    ms = sum(x.elapsed_time(y) for x, y in evs) / steps
    eng.step_events = None
    eng.check_health()
    res = {"model": cfg.name, "recipe": recipe, "layers": cfg.n_layers, "batch": batch, "prompt": prompt, "prefill_tok_s": round(pre),
           "decode_ms_per_step": round(ms, 4), "decode_tok_s": round(batch / (ms / 1e3)),
           "weight_gb": round(eng.model.weight_bytes() / 1e9, 2)}
    for r in reqs:
        eng.abort(r.rid)
    del eng
    import gc
    gc.collect()
    torch.cuda.empty_cache()
    return res


def cut(cfg: ModelConfig, n_layers: int) -> ModelConfig:
    """The first layers of a shape, unlooped."""
    kw = dict(n_layers=n_layers)
    if cfg.has_mixers:
        kw.update(mixers=cfg.mixers[:n_layers], layer_ff=cfg.layer_ff[:n_layers], layer_experts=cfg.layer_experts[:n_layers], loop=None, loop_steps=False)
    return cfg.with_(**kw)
