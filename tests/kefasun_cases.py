"""Engine checks for Kefasun models, run on the CPU back end and on the GPU (bf16 and 32-bit): each takes (device, dtype)."""
from __future__ import annotations

import torch

from llaminar_b200.engine.engine import LLMEngine
from llaminar_b200.engine.sampling import SamplingParams
from llaminar_b200.models.kefasun import weights_from_tensors

from . import kefasun_oracle as oracle
from .pozivik_cases import feed_all, tokens

C, G, L, dense, moe = oracle.chunked_entry, oracle.capped_entry, oracle.latent_entry, oracle.dense, oracle.moe
# name -> (layer list, loop): the three kinds in other orders, unequal layers, every kind of feed-forward behind every kind of mixer,
# loops in every position, sizes that are no multiples of 8 or 16, one head, as many key heads as query heads, keys longer and shorter
# than values, chunks and windows of one token, of a page, and wider than any prompt
MODELS = {
    "kinds": ([C(chunk=20, mlp=moe()), L(window=20), G(softcap=3.0, mlp=moe(4, 1, 24))], {"start": 0, "stop": 2, "times": 2}),
    "order": ([G(heads=6, kv_heads=3, dim=33, vdim=12, rot_dims=6, softcap=20.0), L(heads=5, dim=16, rot_dim=12, vdim=24, kv_rank=33, q_rank=27, window=77, mlp=moe(3, 3, 20)),
               C(heads=3, kv_heads=1, dim=10, vdim=30, rot_dims=10, chunk=64, mlp=None), L(heads=1, window=1000), C(heads=2, kv_heads=2, dim=18, rot_dims=2, chunk=1)], None),
    "loop_middle": ([C(chunk=70), G(mlp=moe(6, 4, 17)), L(window=31, mlp=moe(9, 3, 32)), C(chunk=130, dim=16)], {"start": 1, "stop": 3, "times": 2}),
    "loop_all": ([L(window=65, mlp=None), C(chunk=33, heads=8, kv_heads=2, dim=8, vdim=8, rot_dims=4, mlp=moe(2, 1, 40))], {"start": 0, "stop": 2, "times": 2}),
    "loop_once": ([G(heads=2, kv_heads=1, softcap=50.0), C(chunk=1000, mlp=moe())], {"start": 0, "stop": 1, "times": 1}),
    "loop_end": ([L(window=1, mlp=moe(8, 3, 16)), G(softcap=5.0, mlp=None), C(chunk=65)], {"start": 2, "stop": 3, "times": 3}),
}
# sizes of the tcgen05 kernels (GPU only)
WIDE = ([C(heads=4, kv_heads=2, dim=128, vdim=96, rot_dims=48, chunk=150, mlp=moe(6, 3, 136)), L(heads=20, dim=64, rot_dim=32, vdim=64, kv_rank=128, q_rank=64, window=90, mlp=dense(128)),
         G(heads=6, kv_heads=3, dim=72, vdim=128, rot_dims=72, softcap=12.0, mlp=moe(3, 2, 64)), G(heads=4, kv_heads=4, dim=64, vdim=64, rot_dims=32, softcap=6.0)], {"start": 0, "stop": 2, "times": 2})


def model(name: str, seed: int = 0, **kw):
    layers, loop = WIDE if name == "wide" else MODELS[name]
    return oracle.random_model(layers, seed, loop=loop, **kw)


def engine(m, device, dtype=torch.float32, **kw) -> LLMEngine:
    args = dict(max_batch=4, max_context=640, kv_pages=45, max_prefill_tokens=2048)
    return LLMEngine(weights_from_tensors(m["config"], m["tensors"]), device=device, dtype=dtype, **{**args, **kw})


def tolerance(dtype) -> float:
    return 2e-4 if dtype == torch.float32 else 0.15


CLOSE_CALL = 0.3               # distance of router logits within which 16-bit rounding may choose another expert


def expected(t, m):
    """The oracle's logits, and which positions rest on no close choice of experts."""
    gaps = []
    lg = oracle.forward(t, m, gaps=gaps)
    clear = torch.stack(gaps).min(0).values > CLOSE_CALL if gaps else torch.ones(len(t), dtype=torch.bool)
    return lg, clear


def assert_close(got, want, dtype, what="", rows=None) -> None:
    """Root mean square over the vocabulary of the centred difference, relative to the spread of the logits: its largest value over
    the positions, and over more than a few (a quarter of that) its mean.  ``want``: logits, or what `expected` returns."""
    want, clear = want if isinstance(want, tuple) else (want, torch.ones(len(want), dtype=torch.bool))
    if rows is not None:
        want, clear = want[rows], clear[rows]
    assert torch.isfinite(got).all(), what
    scale = want.double().std()
    if dtype != torch.float32:
        got, want = got[clear.to(got.device)], want[clear]
        if not len(want):
            return
    d = got.double().cpu() - want.double()
    d = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / scale
    assert d.max() < tolerance(dtype) and (len(d) < 8 or d.mean() < tolerance(dtype) / 4), (what, int(d.argmax()), d.max().item(), d.mean().item())


# -- checks ------------------------------------------------------------------------------------------------------------------
def whole_prompt(name, device, dtype):
    m = model(name)
    eng = engine(m, device, dtype)
    for n in (1, 2, 9, 64, 65, 200):
        t = tokens(n, n)
        assert_close(feed_all(eng, t, [n]), expected(t, m), dtype, (name, n))
    assert eng.kv.allocator.n_free == 44                   # every page came back (one is the scratch page)


def portions_and_decoding(name, device, dtype):
    m = model(name, seed=1)
    eng = engine(m, device, dtype)
    t = tokens(230, 3)
    want = expected(t, m)
    for cuts in ([2], [3, 61, 2, 64, 1], [100, 1], [64], [63, 1, 65, 2, 7], [9, 8, 10], [150, 2, 40]):
        assert_close(feed_all(eng, t, cuts), want, dtype, (name, cuts))


def token_by_token(name, device, dtype):
    m = model(name, seed=2)
    eng = engine(m, device, dtype)
    t = tokens(150, 4)
    assert_close(feed_all(eng, t, [1]), expected(t, m), dtype, name)


def mixed_batches(name, device, dtype):
    """Unequal requests side by side, portions beside single tokens, some left out of a step, pages used again by later ones."""
    m = model(name, seed=3)
    eng = engine(m, device, dtype, kv_pages=18)            # room for the live requests only
    rng = torch.Generator().manual_seed(5)
    draw = lambda lo, hi: int(torch.randint(lo, hi, (1,), generator=rng))
    todo = [tokens(n, 10 + i) for i, n in enumerate((150, 3, 97, 210, 1, 64, 129, 40))]
    want = [expected(t, m) for t in todo]
    live, at, nxt = {}, {}, 0
    while nxt < len(todo) or live:
        while nxt < len(todo) and len(live) < 4:
            live[nxt], at[nxt] = eng.open_sequence(), 0
            nxt += 1
        entries, rows = [], []
        for i, r in live.items():
            if len(live) > 1 and draw(0, 5) == 0:
                continue
            n = min(len(todo[i]) - at[i], 1 if draw(0, 2) else draw(2, 40))
            entries.append((r, todo[i][at[i]:at[i] + n], list(range(n))))
            rows += [(i, at[i] + k) for k in range(n)]
            at[i] += n
        if entries:
            got = eng.feed(entries)
            assert_close(got, tuple(torch.stack([want[i][x][k] for i, k in rows]) for x in (0, 1)), dtype, (name, rows[:3]))
        for i in [i for i in live if at[i] == len(todo[i])]:
            eng.close_sequence(live.pop(i))
    assert eng.kv.allocator.n_free == 17


ASKS, ASKED, N = 7, 11, 48


def sharp_model(kind: str, size: int, seed: int = 0):
    """One layer of width N in which a query of token ASKS scores the key of token ASKED far above all others (the rotated values of
    queries and keys are zero, so positions do not matter), so whether that key is visible decides the logits."""
    make = {"attention": lambda: C(heads=2, kv_heads=1, dim=N + 2, vdim=N, rot_dims=2, chunk=size, scale=0.3, mlp=None),
            "attention_2": lambda: G(heads=2, kv_heads=1, dim=N + 2, vdim=N, rot_dims=2, softcap=50.0, scale=0.3, mlp=None),
            "latent_attention": lambda: L(heads=2, window=size, kv_rank=N, q_rank=N, dim=N, vdim=N, scale=0.02, mlp=None)}
    m = oracle.random_model([make[kind]()], seed, width=N)
    t, eye, bf = m["tensors"], torch.eye(N), torch.bfloat16
    one = torch.ones(N, dtype=bf)
    a, b = (oracle.rms_norm(t["embed"][i].float(), 1.0, 1e-5) for i in (ASKS, ASKED))
    t.update({"l0.norm1": one, "l0.norm1b": 3 * one, "l0.mix.g": torch.zeros_like(t["l0.mix.g"])})       # gates of one half
    if kind == "latent_attention":
        rd = m["config"]["layers"][0]["mixer"]["rot_dim"]
        uq = torch.zeros(2, N + rd, N)
        uq[:, :N] = 8 * torch.outer(b, a) / N
        t.update({"l0.mix.dq": eye.to(bf), "l0.mix.uk": torch.cat([eye, eye]).to(bf), "l0.mix.dq.norm": one, "l0.mix.dkv.norm": one,
                  "l0.mix.dkv": torch.cat([eye, torch.zeros(rd, N)]).to(bf), "l0.mix.uq": uq.reshape(-1, N).to(bf), "l0.mix.sink": torch.zeros(2, dtype=bf)})
    else:                                                       # values 0 and 1 rotate: (0, 1) as neighbours and as halves
        q = torch.cat([torch.zeros(2, N), torch.outer(b, a) / N])
        t.update({"l0.mix.q": torch.cat([q, q]).to(bf), "l0.mix.k": torch.cat([torch.zeros(2, N), eye]).to(bf),
                  "l0.mix.q.norm": torch.ones(N + 2, dtype=bf), "l0.mix.k.norm": torch.ones(N + 2, dtype=bf)})
    return m


def ask(start: int, last: int, seed: int) -> list[int]:
    """A sequence whose last token asks for the token at `start`."""
    filler = [i for i in range(97) if i not in (ASKS, ASKED)]
    g = torch.Generator().manual_seed(seed)
    t = [filler[i] for i in torch.randint(0, len(filler), (last + 1,), generator=g).tolist()]
    t[start], t[last] = ASKED, ASKS
    return t


def with_size(m, size):
    layer = m["config"]["layers"][0]
    return {"config": {**m["config"], "layers": [{**layer, "mixer": {**layer["mixer"], "mask": {"size": size}}}]}, "tensors": m["tensors"]}


def check_asked(m, eng, start, last, dtype, what, other=None) -> None:
    """The last token in the prompt, decoded alone, and at the end of a short portion; ``other``: a mask that must give something else."""
    t = ask(start, last, 31 * start + last)
    want = oracle.forward(t, m)
    for cuts in ([last + 1], [max(last, 1), 1], [max(last - 1, 1), 2]):
        assert_close(feed_all(eng, t, cuts)[-1:], want[-1:], dtype, (what, start, last, cuts))
    if other is not None:
        moved = (oracle.forward(t, with_size(m, other))[-1] - want[-1]).std() / want[-1].std()
        assert moved > 2 * tolerance(dtype), ("a mask one token off would not be noticed", what, start, last, moved)


def window_edges(device, dtype):
    """The key that the last token asks for lies near, far back, across page borders, just inside and just outside the window."""
    for window in (64, 65, 100, 130):
        m = sharp_model("latent_attention", window)
        eng = engine(m, device, dtype)
        for back in sorted({1, 2, 63, 64, window - 2, window - 1, window, window + 1}):
            for start in (0, 3, 60, 64):
                other = {window - 1: window - 1, window: window + 1}.get(back)
                check_asked(m, eng, start, start + back, dtype, ("window", window), other)


def chunk_edges(device, dtype):
    """The key that the last token asks for is the first, some or the last of its chunk, or the last or first of the chunk before; the
    last token stands at the start, in the middle and at the end of its chunk."""
    for chunk in (20, 64, 65, 100):
        m = sharp_model("attention", chunk)
        eng = engine(m, device, dtype)
        for n in (1, 2, 4):
            edge = n * chunk
            for last in (edge + 1, edge + chunk // 2, edge + chunk - 1):
                for start in (edge - chunk, edge - 1, edge, min(edge + 3, last - 1)):
                    check_asked(m, eng, start, last, dtype, ("chunk", chunk))
            # one token more or less per chunk would move the border across the key that is asked for
            check_asked(m, eng, edge, edge + chunk - 1, dtype, ("first of the chunk", chunk), chunk + 1)
            check_asked(m, eng, edge - 1, edge, dtype, ("last of the chunk before", chunk), chunk + 1)
            check_asked(m, eng, edge - 1, edge + chunk // 2, dtype, ("chunk before", chunk), 10 ** 6)


def far_keys(device, dtype):
    """Causal attention finds a key anywhere, in other pages and hundreds of tokens back."""
    m = sharp_model("attention_2", 0)
    eng = engine(m, device, dtype)
    for start, last in ((0, 1), (0, 64), (63, 64), (64, 127), (1, 300), (130, 333), (0, 600), (5, 575)):
        t = ask(start, last, 7)
        want = oracle.forward(t, m)
        blind = oracle.forward([t[0] if i == start else x for i, x in enumerate(t)] if start else [x if i else (t[1] if t[1] != ASKS else 12) for i, x in enumerate(t)], m)
        assert (blind[-1] - want[-1]).std() / want[-1].std() > 2 * tolerance(dtype)
        check_asked(m, eng, start, last, dtype, "far")


def sinks_matter(device, dtype):
    """A sink that takes most of the weight, and one that takes none; the first tokens of a sequence feel it most."""
    for sink in (-30.0, 0.0, 6.0):
        m = model("loop_all", seed=6, sink_shift=sink)
        eng = engine(m, device, dtype)
        t = tokens(140, 8)
        want = expected(t, m)
        assert_close(feed_all(eng, t, [140]), want, dtype, sink)
        assert_close(feed_all(eng, t, [1]), want, dtype, sink)


def long_decoding(device, dtype):
    m = model("kinds", seed=7)
    eng = engine(m, device, dtype)
    t = tokens(600, 9)
    assert_close(feed_all(eng, t, [70, 1])[::7], expected(t, m), dtype, rows=slice(None, None, 7))


def greedy_generation(device, dtype):
    """Through add_request / step: batches of unequal prompts, more requests than lanes, pages used again, chunked prefill."""
    m = model("order", seed=8, gain=1.3)
    prompts = [tokens(n, 20 + n) for n in (5, 70, 130, 64, 1, 33)]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    outs = engine(m, device, dtype).generate(prompts, sp)
    small = engine(m, device, dtype, kv_pages=12, max_prefill_tokens=48, max_batch=2)
    assert small.generate(prompts, sp) == outs or dtype != torch.float32
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        lg = oracle.forward(p + o, m)[len(p) - 1:-1]
        top = lg.max(-1).values - lg.gather(1, torch.tensor(o)[:, None])[:, 0]
        assert (top < 3 * tolerance(dtype) * lg.std()).all(), top.max()      # every emitted token is (nearly) the oracle's best


def prefix_cache_reuse(device, dtype):
    from llaminar_b200.engine.prefix_cache import PrefixCache, PrefixCacheConfig
    m = model("loop_middle", seed=9)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    plain = engine(m, device, dtype)
    cached = engine(m, device, dtype, prefix_cache=PrefixCache(PrefixCacheConfig(), fingerprint="test"))
    base = tokens(140, 30)
    for tail in ([1, 2, 3], [4], [1, 2, 3]):
        a, b = plain.generate([base + tail], sp), cached.generate([base + tail], sp)
        assert a == b or dtype != torch.float32
    assert cached.stats["prefix_hit_tokens"] >= 128
    page = cached.kv.export_page(1)
    before = [l[1].clone() for l in cached.kv.layers]
    cached.kv.import_page(1, page)
    assert all(torch.equal(x, l[1]) for x, l in zip(before, cached.kv.layers))


def preemption(device, dtype):
    """A pool too small for both: one sequence is preempted, comes back and continues with the same tokens."""
    m = model("kinds", seed=10)
    prompts = [tokens(60, 40), tokens(62, 41)]
    sp = SamplingParams(temperature=0.0, max_tokens=80, ignore_eos=True)
    outs = engine(m, device, dtype).generate(prompts, sp)
    eng = engine(m, device, dtype, kv_pages=5)
    got = eng.generate(prompts, sp)
    assert eng.stats["preemptions"] > 0 and all(len(o) == 80 for o in got)
    assert got == outs or dtype != torch.float32


ENGINE_CHECKS = ["window_edges", "chunk_edges", "far_keys", "sinks_matter", "long_decoding", "greedy_generation", "prefix_cache_reuse", "preemption"]
