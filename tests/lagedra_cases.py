"""Engine checks for Lagedra models, run on the CPU back end and on the GPU (bf16 and 32-bit): each takes (device, dtype)."""
from __future__ import annotations

import torch

from llaminar_b200.engine.engine import LLMEngine
from llaminar_b200.engine.sampling import SamplingParams
from llaminar_b200.models.lagedra import weights_from_tensors

from . import lagedra_oracle as oracle
from .kefasun_cases import tolerance
from .pozivik_cases import feed_all, tokens

A, L, dense, moe = oracle.attention_entry, oracle.lightning_entry, oracle.dense, oracle.moe
# name -> layer list: both mixers in several orders, every kind of feed-forward (or none) behind either, unequal layers, value mixing that
# starts late, pauses or is absent, filters of one to seven taps, sizes that are no multiples of 8, one head, as many key heads as query
# heads, keys longer and shorter than values, windows of one token, of a page, wider than any prompt and none, groups of one expert
MODELS = {
    "kinds": [L(), A(mlp=moe()), A(conv=3, mlp=dense(72)), L(heads=2, dim=16, vdim=40, mlp=moe(8, 3, 24, 4, 2, 0.8))],
    "order": [A(heads=6, kv_heads=3, dim=33, vdim=12, rot_dims=6, window=64, conv=2, v_mix=False, mlp=None), L(heads=1, dim=60, vdim=33, decay=(0.97,), mlp=moe(6, 2, 20, 1, 1)),
              A(heads=3, kv_heads=1, dim=10, vdim=30, rot_dims=10, window=77, conv=7, softcap=2.0, scaling=None), A(heads=2, kv_heads=1, dim=18, vdim=30, rot_dims=2, window=1, conv=1, mlp=moe(6, 1, 17, 6, 3)),
              L(mlp=None), A(heads=2, kv_heads=1, dim=40, vdim=30, window=1000, conv=5, softcap=None, scale=0.06)],
    "pauses": [A(window=31, v_mix=False), A(window=65), A(window=130, v_mix=False, mlp=moe(4, 4, 17, 2, 2)), A(heads=8, kv_heads=2, dim=8, window=33, rot_dims=8), L(heads=3, decay=(1.0, 0.2, 0.9))],
    "recurrent": [L(heads=2, dim=30, vdim=8), L(heads=3, dim=36, vdim=7, mlp=dense(33))],
    "attending": [A(heads=1, kv_heads=1, window=None, mlp=None), A(heads=4, kv_heads=1, window=63, conv=2)],
}
# sizes of the tcgen05 kernels (GPU only)
WIDE = [L(heads=3, dim=128, vdim=256, mlp=dense(256)), A(heads=8, kv_heads=2, dim=128, vdim=96, rot_dims=128, window=90, mlp=moe(8, 4, 64, 4, 3)), L(heads=2, dim=64, vdim=320, mlp=moe(8, 2, 136, 2, 1)),
        A(heads=4, kv_heads=2, dim=64, vdim=96, rot_dims=32, window=300, conv=3)]


def model(name: str, seed: int = 0, **kw):
    return oracle.random_model(WIDE if name == "wide" else MODELS[name], seed, **kw)


def engine(m, device, dtype=torch.float32, **kw) -> LLMEngine:
    args = dict(max_batch=4, max_context=640, kv_pages=45, max_prefill_tokens=2048)
    return LLMEngine(weights_from_tensors(m["config"], m["tensors"]), device=device, dtype=dtype, **{**args, **kw})


def expected(t, m, dt=torch.float64):
    """The oracle's logits, and how far every position's choices of experts are from turning out otherwise (None: all are certain);
    zero also where one of the few tokens before hangs in the balance, which the mixers hand on."""
    gaps = []
    lg = oracle.forward(t, m, dt=dt, gaps=gaps)
    gap = torch.stack(gaps).min(0).values if gaps else torch.full((len(t),), float("inf"))
    for p in (gap < 0.05).nonzero().flatten().tolist():
        gap[p:p + 8] = 0.0
    return lg, None if bool(gap.isinf().all()) else gap


CLOSE_CALL = 0.3               # distance of router logits within which 16-bit rounding may choose another expert


def assert_close(got, want, dtype, what="", rows=None) -> None:
    """Root mean square over the vocabulary of the centred difference, relative to the spread of the logits: its largest value over
    the positions and (a quarter of that) its mean.  ``want``: logits, or what `expected` returns; in 16 bits positions that rest on a
    close choice of experts are left out, and one in ten others may have seen such a position through a mixer."""
    want, gap = want if isinstance(want, tuple) else (want, None)
    if rows is not None:
        want, gap = want[rows], None if gap is None else gap[rows]
    assert torch.isfinite(got).all(), what
    scale, tol = want.double().std(), tolerance(dtype)
    d = got.double().cpu() - want.double()
    d = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / scale
    if gap is not None and dtype != torch.float32:
        d = d[gap > CLOSE_CALL]
        d = d.sort().values[:len(d) - len(d) // 10]
    assert not len(d) or (d.max() < tol and (len(d) < 8 or d.mean() < tol / 4)), (what, int(d.argmax()), d.max().item(), d.mean().item())


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
    for cuts in ([2], [3, 61, 2, 64, 1], [100, 1], [64], [63, 1, 65, 2, 7], [9, 8, 10], [150, 2, 40], [1, 128, 3, 1, 5]):
        assert_close(feed_all(eng, t, cuts), want, dtype, (name, cuts))


def token_by_token(name, device, dtype):
    m = model(name, seed=2)
    eng = engine(m, device, dtype)
    t = tokens(150, 4)
    assert_close(feed_all(eng, t, [1]), expected(t, m), dtype, name)


def mixed_batches(name, device, dtype):
    """Unequal requests side by side, portions beside single tokens, some left out of a step, pages and slots used again by later ones."""
    m = model(name, seed=3)
    eng = engine(m, device, dtype, kv_pages=18)            # room for the live requests only
    rng = torch.Generator().manual_seed(5)
    draw = lambda lo, hi: int(torch.randint(lo, hi, (1,), generator=rng))
    todo = [tokens(n, 10 + i) for i, n in enumerate((150, 3, 97, 210, 1, 64, 129, 40))]
    want = [expected(t, m) for t in todo]
    live, at, nxt, got, rows = {}, {}, 0, [], []
    while nxt < len(todo) or live:
        while nxt < len(todo) and len(live) < 4:
            live[nxt], at[nxt] = eng.open_sequence(), 0
            nxt += 1
        entries = []
        for i, r in live.items():
            if len(live) > 1 and draw(0, 5) == 0:
                continue
            n = min(len(todo[i]) - at[i], 1 if draw(0, 2) else draw(2, 40))
            entries.append((r, todo[i][at[i]:at[i] + n], list(range(n))))
            rows += [(i, at[i] + k) for k in range(n)]
            at[i] += n
        if entries:
            got.append(eng.feed(entries).clone())
        for i in [i for i in live if at[i] == len(todo[i])]:
            eng.close_sequence(live.pop(i))
    pick = lambda x: None if want[0][x] is None else torch.stack([want[i][x][k] for i, k in rows])
    assert_close(torch.cat(got), (pick(0), pick(1)), dtype, name)
    assert eng.kv.allocator.n_free == 17 and len(eng.kv.hybrid.free) == 4


ASKS, ASKED, N = 7, 11, 48


def plain_layer(layer, seed: int):
    """One layer of width N without position vectors, whose output stands beside the embedding with equal weight."""
    m = oracle.random_model([layer], seed, width=N)
    t, bf = m["tensors"], torch.bfloat16
    t.update({"pos": torch.zeros_like(t["pos"]), "l0.norm1": torch.tensor(1.0, dtype=bf), "l0.dwa": torch.tensor([0.5, 1.0], dtype=bf)})
    a, b = (oracle.scalar_norm(t["embed"][i].float(), 1.0, 1e-5) for i in (ASKS, ASKED))
    return m, a, b


def sharp_model(window: int, seed: int = 0):
    """A query of token ASKS scores the key of token ASKED far above all others (the rotated values of queries and keys are zero and the
    filters let the newest row through, so positions do not matter): whether that key is visible decides the logits."""
    m, a, b = plain_layer(A(heads=2, kv_heads=1, dim=N + 2, vdim=N, rot_dims=2, window=window, conv=3, softcap=50.0, scale=0.3, scaling=None, v_mix=False, mlp=None), seed)
    t, bf = m["tensors"], torch.bfloat16
    q = torch.cat([torch.zeros(2, N), torch.outer(b, a) / N])
    t.update({"l0.mix.q": torch.cat([q, q]).to(bf), "l0.mix.k": torch.cat([torch.zeros(2, N), torch.eye(N)]).to(bf), "l0.mix.temp": torch.ones(2, dtype=bf),
              "l0.mix.o": 3 * t["l0.mix.o"]})
    for x in "qkv":
        t[f"l0.mix.{x}.conv"] = torch.tensor([0.0, 0.0, 1.0], dtype=bf).expand(t[f"l0.mix.{x}.conv"].shape[0], 3).clone()
    return m


def memory_model(seed: int = 0):
    """Lightning attention in which token ASKED leaves a state that takes long to fade; with it the tokens that leave next to none (those
    whose embeddings point away from its own, so that silu closes)."""
    m, a, b = plain_layer(L(heads=2, dim=16, vdim=N, decay=(0.9995, 0.998), mlp=None), seed)
    one = torch.ones(32)
    m["tensors"].update({"l0.mix.q": (torch.outer(one, a) * 4 / N).bfloat16(), "l0.mix.k": (torch.outer(one, b) * 160 / N).bfloat16(), "l0.mix.o": 3 * m["tensors"]["l0.mix.o"]})
    return m, [i for i in range(97) if float(m["tensors"]["embed"][i].float() @ b) < -3]


def ask(start: int, last: int, seed: int, filler=None) -> list[int]:
    """A sequence whose last token asks for the token at `start`; ``filler``: the tokens between."""
    filler = [i for i in filler or range(97) if i not in (ASKS, ASKED)]
    g = torch.Generator().manual_seed(seed)
    t = [filler[i] for i in torch.randint(0, len(filler), (last + 1,), generator=g).tolist()]
    t[start], t[last] = ASKED, ASKS
    return t


def with_window(m, size):
    layer = m["config"]["layers"][0]
    return {"config": {**m["config"], "layers": [{**layer, "mixer": {**layer["mixer"], "mask": {"size": size}}}]}, "tensors": m["tensors"]}


def matters(a, b, dtype) -> bool:
    """Whether two rows of logits differ by more than any check lets pass."""
    d = a - b
    return bool((d - d.mean()).pow(2).mean().sqrt() / b.std() > 2 * tolerance(dtype))


def check_asked(m, eng, start, last, dtype, what, other=None, t=None) -> None:
    """The last token in the prompt, decoded alone, and at the end of a short portion; ``other``: a window that must give something else."""
    t = t or ask(start, last, 31 * start + last)
    want = oracle.forward(t, m)
    for cuts in ([last + 1], [max(last, 1), 1], [max(last - 1, 1), 2]):
        assert_close(feed_all(eng, t, cuts)[-1:], want[-1:], dtype, (what, start, last, cuts))
    if other is not None:
        assert matters(oracle.forward(t, with_window(m, other))[-1], want[-1], dtype), ("a window one token off would not be noticed", what, start, last)


def window_edges(device, dtype):
    """The key that the last token asks for lies near, far back, across page borders, just inside and just outside the window."""
    for window in (30, 64, 65, 130):
        m = sharp_model(window)
        eng = engine(m, device, dtype)
        for back in sorted({1, 2, 63, 64, window - 2, window - 1, window, window + 1}):
            for start in (0, 3, 60, 64):
                other = {window - 1: window - 1, window: window + 1}.get(back)
                check_asked(m, eng, start, start + back, dtype, ("window", window), other)


def far_memory(device, dtype):
    """The recurrence finds a token in other pages and chunks and hundreds of tokens back, whatever was cut in between."""
    m, filler = memory_model()
    eng = engine(m, device, dtype)
    for start, last in ((0, 1), (0, 64), (63, 64), (127, 128), (1, 300), (130, 333), (0, 600), (5, 575)):
        t = ask(start, last, 7, filler)
        assert matters(oracle.forward([filler[0] if x == ASKED else x for x in t], m)[-1], oracle.forward(t, m)[-1], dtype)
        check_asked(m, eng, start, last, dtype, "far", t=t)


def oldest_tap(device, dtype):
    """Filters that pass only their oldest row: the first rows of a sequence are zeros, the state matters behind every cut."""
    for taps in (1, 2, 3, 4, 6):
        m = oracle.random_model([A(conv=taps, v_mix=False, window=40), A(conv=taps, window=7, mlp=None)], seed=taps)
        for name, x in m["tensors"].items():
            if name.endswith(".conv"):
                m["tensors"][name] = (torch.arange(taps) == 0).to(torch.bfloat16).expand_as(x).clone()
        t = tokens(90, 5)
        want = oracle.forward(t, m)
        eng = engine(m, device, dtype)
        for cuts in ([90], [1], [2], [3, 1, 4], [5, 60, 1], [taps, 1], [max(1, taps - 1), 2]):
            assert_close(feed_all(eng, t, cuts), want, dtype, (taps, cuts))


def used_slots(device, dtype):
    """A slot's former owner leaves nothing behind, in prompts and when the first tokens come one by one."""
    m = model("kinds", seed=6)
    eng = engine(m, device, dtype, max_batch=1, kv_pages=12)
    t = tokens(40, 8)
    want = expected(t, m)
    for cuts in ([40], [1], [2], [1, 3]):
        feed_all(eng, tokens(300, 9), [299, 1])
        assert_close(feed_all(eng, t, cuts), want, dtype, cuts)


def positions_end(device, dtype):
    """The table of position vectors bounds a sequence."""
    m = model("attending", seed=4, max_positions=70)
    eng = engine(m, device, dtype)
    t = tokens(70, 3)
    assert_close(feed_all(eng, t, [60, 9, 1]), expected(t, m), dtype)
    r = eng.open_sequence()
    eng.feed([(r, t, [])])
    try:
        eng.feed([(r, [1], [])])
        raise AssertionError("a position without a vector was accepted")
    except ValueError:
        eng.close_sequence(r)


def long_decoding(device, dtype):
    m = model("kinds", seed=7)
    eng = engine(m, device, dtype)
    t = tokens(600, 9)
    assert_close(feed_all(eng, t, [70, 1])[::7], expected(t, m), dtype, rows=slice(None, None, 7))


def greedy_generation(device, dtype):
    """Through add_request / step: batches of unequal prompts, more requests than lanes, pages used again, chunked prefill."""
    m = model("kinds", seed=8)
    prompts = [tokens(n, 20 + n) for n in (5, 70, 130, 64, 1, 33)]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    outs = engine(m, device, dtype).generate(prompts, sp)
    small = engine(m, device, dtype, kv_pages=12, max_prefill_tokens=48, max_batch=2)
    assert small.generate(prompts, sp) == outs or dtype != torch.float32
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        lg, gap = (x[len(p) - 1:-1] for x in expected(p + o, m))
        top = lg.max(-1).values - lg.gather(1, torch.tensor(o)[:, None])[:, 0]
        top = top[gap > CLOSE_CALL] if dtype != torch.float32 else top
        assert (top < 3 * tolerance(dtype) * lg.std()).all(), top.max()      # every emitted token is (nearly) the oracle's best


def prefix_cache_reuse(device, dtype):
    from llaminar_b200.engine.prefix_cache import PrefixCache, PrefixCacheConfig
    m = model("pauses", seed=9)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    plain = engine(m, device, dtype)
    cached = engine(m, device, dtype, prefix_cache=PrefixCache(PrefixCacheConfig(), fingerprint="test"))
    base = tokens(140, 30)
    for tail in ([1, 2, 3], [4], [1, 2, 3]):
        a, b = plain.generate([base + tail], sp), cached.generate([base + tail], sp)
        assert a == b or dtype != torch.float32
    assert cached.stats["prefix_hit_tokens"] >= 128


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


ENGINE_CHECKS = ["window_edges", "far_memory", "oldest_tap", "used_slots", "positions_end", "long_decoding", "greedy_generation", "prefix_cache_reuse", "preemption"]
