"""Engine checks for Pozivik models, run on the CPU back end and on the GPU (bf16 and 32-bit): each takes (device, dtype)."""
from __future__ import annotations

import torch

from llaminar_b200.engine.engine import LLMEngine
from llaminar_b200.engine.sampling import SamplingParams
from llaminar_b200.models.pozivik import weights_from_tensors

from . import pozivik_oracle as oracle

YARN = {"factor": 3.0, "original": 64, "fast": 16.0, "slow": 1.0}
E = oracle.layer_entry
# name -> (layer list, loop): unequal layers, no feed-forward, loops in every position, sizes that are no multiples of 8 or 16,
# one head, windows of one page, of one token, and wider than any prompt
MODELS = {
    "mixed": ([E(window=20), E(heads=5, dim=16, rot_dim=12, vdim=24, kv_rank=33, q_rank=27, window=77, scaling=YARN), E(ff=None, window=64), E(heads=1, window=1000)], None),
    "loop_middle": ([E(window=70, scaling=YARN), E(window=31), E(ff=40, window=130)], {"start": 1, "stop": 2, "times": 3}),
    "loop_all": ([E(window=65), E(heads=2, dim=8, rot_dim=16, vdim=8, kv_rank=24, q_rank=16, window=5)], {"start": 0, "stop": 2, "times": 2}),
    "loop_once": ([E(window=1), E(window=63), E(window=200, base=50.0)], {"start": 0, "stop": 1, "times": 1}),
    "loop_end": ([E(window=33), E(window=64, ff=None)], {"start": 1, "stop": 2, "times": 2}),
}
# sizes of the tcgen05 kernels (GPU only)
WIDE = ([E(heads=20, dim=64, rot_dim=32, vdim=64, kv_rank=128, q_rank=64, window=90, ff=128, scaling=YARN),
         E(heads=6, dim=32, rot_dim=16, vdim=48, kv_rank=256, q_rank=48, window=300, ff=96)], {"start": 1, "stop": 2, "times": 2})


def model(name: str, seed: int = 0, width: int = 48, **kw):
    layers, loop = WIDE if name == "wide" else MODELS[name]
    return oracle.random_model(seed, layers=layers, loop=loop, width=width, **kw)


def engine(m, device, dtype=torch.float32, **kw) -> LLMEngine:
    args = dict(max_batch=4, max_context=640, kv_pages=45, max_prefill_tokens=2048)
    return LLMEngine(weights_from_tensors(m["config"], m["tensors"]), device=device, dtype=dtype, **{**args, **kw})


def tokens(n: int, seed: int, vocab: int = 97) -> list[int]:
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def tolerance(dtype) -> float:
    return 2e-4 if dtype == torch.float32 else 0.25


def assert_close(got, want, dtype, what="") -> None:
    """Root mean square over the vocabulary of the centred difference, relative to the spread of the logits: its largest value
    over the positions, and (a quarter of that) its mean."""
    d = got.double().cpu() - want.double()
    d = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().std()
    assert torch.isfinite(d).all() and d.max() < tolerance(dtype) and d.mean() < tolerance(dtype) / 4, (what, int(d.argmax()), d.max().item(), d.mean().item())


def feed_all(eng, toks, cuts) -> torch.Tensor:
    """Logits of every position, the sequence fed in portions of the given sizes (the last one repeats)."""
    r, out, at, i = eng.open_sequence(), [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(eng.feed([(r, toks[at:at + n], list(range(n)))]).clone())
        at, i = at + n, i + 1
    eng.close_sequence(r)
    return torch.cat(out)


# -- checks ------------------------------------------------------------------------------------------------------------------
def whole_prompt(name, device, dtype):
    m = model(name)
    eng = engine(m, device, dtype)
    for n in (1, 2, 9, 64, 65, 200):
        t = tokens(n, n)
        assert_close(feed_all(eng, t, [n]), oracle.forward(t, m), dtype, (name, n))
    assert eng.kv.allocator.n_free == 44                   # every page came back (one is the scratch page)


def portions_and_decoding(name, device, dtype):
    m = model(name, seed=1)
    eng = engine(m, device, dtype)
    t = tokens(230, 3)
    want = oracle.forward(t, m)
    for cuts in ([2], [3, 61, 2, 64, 1], [100, 1], [64], [63, 1, 65, 2, 7], [9, 8, 10]):
        assert_close(feed_all(eng, t, cuts), want, dtype, (name, cuts))


def token_by_token(name, device, dtype):
    m = model(name, seed=2)
    eng = engine(m, device, dtype)
    t = tokens(150, 4)
    assert_close(feed_all(eng, t, [1]), oracle.forward(t, m), dtype, name)


def mixed_batches(name, device, dtype):
    """Unequal requests side by side, portions beside single tokens, some left out of a step, pages used again by later ones."""
    m = model(name, seed=3)
    eng = engine(m, device, dtype, kv_pages=18)            # room for the live requests only
    rng = torch.Generator().manual_seed(5)
    draw = lambda lo, hi: int(torch.randint(lo, hi, (1,), generator=rng))
    todo = [tokens(n, 10 + i) for i, n in enumerate((150, 3, 97, 210, 1, 64, 129, 40))]
    want = [oracle.forward(t, m) for t in todo]
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
            assert_close(got, torch.stack([want[i][k] for i, k in rows]), dtype, (name, rows[:3]))
        for i in [i for i in live if at[i] == len(todo[i])]:
            eng.close_sequence(live.pop(i))
    assert eng.kv.allocator.n_free == 17


ASKS, ASKED = 7, 11


def sharp_model(window: int, seed: int = 0):
    """One layer in which a query of token ASKS scores the key of token ASKED far above all others (no position in the scores:
    the rotated parts are zero), so whether that key is visible decides the logits."""
    layers = [E(heads=2, window=window, kv_rank=48, q_rank=48, dim=48, vdim=48, ff=None, scale=0.02)]
    m = oracle.random_model(seed, layers=layers, width=48, vocab=97)
    t, mix, eye = m["tensors"], layers[0]["mixer"], torch.eye(48)
    zero, one = torch.zeros(48, dtype=torch.bfloat16), torch.ones(48, dtype=torch.bfloat16)
    t.update({"l0.norm1": zero, "embed.norm": zero, "l0.norm1b": zero, "l0.mix.dq.norm": one, "l0.mix.dkv.norm": one})
    a, b = (oracle.rms_divide(t["embed"][i].float(), 1e-5) for i in (ASKS, ASKED))
    uq = torch.zeros(2, 48 + mix["rot_dim"], 48)
    uq[:, :48] = 8 * torch.outer(b, a) / 48                     # |a|^2 = 48: the query of ASKS is 8 b
    t["l0.mix.dq"], t["l0.mix.uk"] = eye.to(torch.bfloat16), torch.cat([eye, eye]).to(torch.bfloat16)
    t["l0.mix.dkv"] = torch.cat([eye, torch.zeros(mix["rot_dim"], 48)]).to(torch.bfloat16)
    t["l0.mix.uq"] = uq.reshape(-1, 48).to(torch.bfloat16)
    t["l0.mix.sink"] = torch.zeros(2, dtype=torch.bfloat16)
    return m


def far_keys_and_window_edges(device, dtype):
    """The key that the last token asks for lies near, far back, across page borders, just inside and just outside the window;
    the last token is part of the prompt or decoded alone.  The oracle must tell the two sides of the edge apart clearly."""
    filler = [i for i in range(97) if i not in (ASKS, ASKED)]
    for window in (64, 65, 100, 130):
        m = sharp_model(window)
        eng = engine(m, device, dtype)
        g = torch.Generator().manual_seed(window)
        for back in sorted({1, 2, 63, 64, window - 2, window - 1, window, window + 1}):
            for start in (0, 3, 60, 64):
                n = start + back + 1
                t = [filler[i] for i in torch.randint(0, len(filler), (n,), generator=g).tolist()]
                t[start], t[n - 1] = ASKED, ASKS
                want = oracle.forward(t, m)
                assert_close(feed_all(eng, t, [n])[-1:], want[-1:], dtype, ("prompt", window, back, start))
                assert_close(feed_all(eng, t, [n - 1, 1])[-1:], want[-1:], dtype, ("decoded", window, back, start))
                if back in (window - 1, window):
                    layer = m["config"]["layers"][0]
                    other = {**layer, "mixer": {**layer["mixer"], "mask": {"size": window + (1 if back == window else -1)}}}
                    moved = oracle.forward(t, {"config": {**m["config"], "layers": [other]}, "tensors": m["tensors"]})[-1] - want[-1]
                    assert (moved.std() / want[-1].std()) > tolerance(dtype), "a window one token off would not be noticed"      # four times what passes for one row


def sinks_matter(device, dtype):
    """A sink that takes most of the weight, and one that takes none; the first tokens of a sequence feel it most."""
    for sink in (-30.0, 0.0, 6.0):
        m = model("loop_middle", seed=6, sink_shift=sink)
        eng = engine(m, device, dtype)
        t = tokens(140, 8)
        want = oracle.forward(t, m)
        assert_close(feed_all(eng, t, [140]), want, dtype, sink)
        assert_close(feed_all(eng, t, [1]), want, dtype, sink)


def long_decoding(device, dtype):
    m = model("loop_all", seed=7)
    eng = engine(m, device, dtype)
    t = tokens(600, 9)
    want = oracle.forward(t, m)
    assert_close(feed_all(eng, t, [70, 1])[::7], want[::7], dtype)


def greedy_generation(device, dtype):
    """Through add_request / step: batches of unequal prompts, more requests than lanes, pages used again, chunked prefill."""
    m = model("mixed", seed=8, gain=1.3)
    prompts = [tokens(n, 20 + n) for n in (5, 70, 130, 64, 1, 33)]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    outs = engine(m, device, dtype).generate(prompts, sp)
    small = engine(m, device, dtype, kv_pages=12, max_prefill_tokens=48, max_batch=2)
    assert small.generate(prompts, sp) == outs or dtype != torch.float32
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        lg = oracle.forward(p + o, m)[len(p) - 1:-1]
        top = lg.max(-1).values - lg.gather(1, torch.tensor(o)[:, None])[:, 0]
        assert (top < tolerance(dtype) * lg.std()).all(), top.max()      # every emitted token is (nearly) the oracle's best


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
    m = model("mixed", seed=10)
    prompts = [tokens(60, 40), tokens(62, 41)]
    sp = SamplingParams(temperature=0.0, max_tokens=80, ignore_eos=True)
    outs = engine(m, device, dtype).generate(prompts, sp)
    eng = engine(m, device, dtype, kv_pages=5)
    got = eng.generate(prompts, sp)
    assert eng.stats["preemptions"] > 0 and all(len(o) == 80 for o in got)
    assert got == outs or dtype != torch.float32
