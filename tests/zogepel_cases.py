"""Engine checks for Zogepel models, run on the CPU back end and on the GPU (bf16 and 32-bit): each takes (device, dtype)."""
from __future__ import annotations

import torch

from llaminar_b200.engine.engine import LLMEngine
from llaminar_b200.engine.sampling import SamplingParams
from llaminar_b200.models.zogepel import weights_from_tensors

from . import zogepel_oracle as oracle

M, P = oracle.mlstm_layer, oracle.parallel_layer
# name -> layer list: unequal layers of both kinds, no feed-forward, sizes that are no multiples of 8 or 16, one head, as many key
# heads as query heads, rotation of all, some and two values of a head, decays near 0 and 1, windows of one page, of one token and
# wider than any prompt
MODELS = {
    "both": [M(), P(), M(heads=2, dim=16, vdim=40, cap=4.0), P(heads=6, kv_heads=3, dim=16, window=77, r_heads=2, r_dim=32, r_vdim=16, r_rot=32, decay=[0.997, 0.98])],
    "lstm": [M(heads=1, dim=30, vdim=22, ff=None), M(heads=5, dim=8, vdim=8, cap=30.0, ff=40)],
    "parallel": [P(heads=2, kv_heads=2, dim=33, window=64, r_heads=1, r_dim=9, r_vdim=13, r_rot=2, decay=[0.5], ff=None), P(heads=5, kv_heads=1, window=1, scale=0.5),
                 P(window=1000, r_heads=4, r_dim=16, r_vdim=64, r_rot=16, decay=[0.999, 0.9, 1.0, 0.05])],
    "edges": [P(window=65, ff=32), M(ff=24), P(window=130, heads=3, kv_heads=1, dim=64, ff=72)],
}
# head sizes of the tensor-core kernels, chunks of several tiles (GPU only)
WIDE = [M(heads=3, dim=64, vdim=128, ff=128), P(heads=8, kv_heads=2, dim=128, window=200, r_heads=2, r_dim=128, r_vdim=96, r_rot=64, ff=64),
        P(heads=4, kv_heads=4, dim=64, window=90, r_heads=3, r_dim=48, r_vdim=256, r_rot=48), M(heads=2, dim=128, vdim=272, cap=8.0)]


def model(name: str, seed: int = 0, width: int = 48, **kw):
    return oracle.random_model(seed, layers=WIDE if name == "wide" else MODELS[name], width=width, **kw)


def engine(m, device, dtype=torch.float32, **kw) -> LLMEngine:
    args = dict(max_batch=4, max_context=640, kv_pages=45, max_prefill_tokens=2048)
    return LLMEngine(weights_from_tensors(m["config"], m["tensors"]), device=device, dtype=dtype, **{**args, **kw})


def tokens(n: int, seed: int, vocab: int = 97) -> list[int]:
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def tolerance(dtype) -> float:
    return 2e-4 if dtype == torch.float32 else 0.1


def assert_close(got, want, dtype, what="", factor=1.0) -> None:
    """Root mean square over the vocabulary of the centred difference, relative to the spread of the logits: its largest value
    over the positions, and over more than a few its mean."""
    d = got.double().cpu() - want.double()
    d = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().std()
    ok = torch.isfinite(d).all() and d.max() < 1.5 * factor * tolerance(dtype) and (len(d) < 8 or d.mean() < factor * tolerance(dtype) / 5)
    assert ok, (what, int(d.argmax()), d.max().item(), d.mean().item())


def feed_all(eng, toks, cuts) -> torch.Tensor:
    """Logits of every position, the sequence fed in portions of the given sizes (the last one repeats)."""
    r, out, at, i = eng.open_sequence(), [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(eng.feed([(r, toks[at:at + n], list(range(n)))]).clone())
        at, i = at + n, i + 1
    eng.close_sequence(r)
    return torch.cat(out)


def all_free(eng) -> bool:
    """Every page (but the scratch page) and every state slot is free."""
    return eng.kv.allocator.n_free == eng.kv.n_pages - 1 and len(eng.kv.hybrid.free) == eng.kv.hybrid.n_slots


# -- checks ------------------------------------------------------------------------------------------------------------------
def whole_prompt(name, device, dtype):
    m = model(name)
    eng = engine(m, device, dtype)
    for n in (1, 2, 9, 64, 65, 200):
        t = tokens(n, n)
        assert_close(feed_all(eng, t, [n]), oracle.forward(t, m), dtype, (name, n))
    assert all_free(eng)


def portions_and_decoding(name, device, dtype):
    m = model(name, seed=1)
    eng = engine(m, device, dtype)
    t = tokens(230, 3)
    want = oracle.forward(t, m)
    for cuts in ([2], [3, 61, 2, 64, 1], [100, 1], [64], [63, 1, 65, 2, 7], [9, 8, 10], [129, 127 - 30]):
        assert_close(feed_all(eng, t, cuts), want, dtype, (name, cuts))


def token_by_token(name, device, dtype):
    m = model(name, seed=2)
    eng = engine(m, device, dtype)
    t = tokens(150, 4)
    assert_close(feed_all(eng, t, [1]), oracle.forward(t, m), dtype, name)


def mixed_batches(name, device, dtype):
    """Unequal requests side by side, portions beside single tokens, some left out of a step, pages and slots used again by later ones."""
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
    assert all_free(eng)


ASKS, ASKED = 7, 11
SHARP = 0.5                    # where one key decides: half the tolerance, and a mistake moves the logits by more than all of it


def sharp_attention(window: int, seed: int = 0):
    """One layer in which a query of token ASKS scores the key of token ASKED far above all others, so whether that key is visible
    decides the logits; the retention beside it forgets at once."""
    layers = [P(heads=2, kv_heads=1, dim=48, window=window, scale=0.15, r_heads=1, r_dim=8, r_vdim=8, r_rot=8, decay=[0.0], ff=None)]
    m = oracle.random_model(seed, layers=layers, width=48, side_dim=4)
    t = m["tensors"]
    a, b = (oracle.rms_divide(t["embed"][i].float(), 1e-9) for i in (ASKS, ASKED))
    one, zero = torch.ones(48, dtype=torch.bfloat16), torch.zeros(48, dtype=torch.bfloat16)
    t["l0.mix.left.k"] = torch.eye(48).to(torch.bfloat16)
    q = torch.outer(b, a) + 0.02 * torch.randn(48, 48, generator=torch.Generator().manual_seed(1))
    t["l0.mix.left.q"] = torch.cat([q, q]).to(torch.bfloat16)                 # the query of ASKS points along b
    t["l0.mix.left.q.norm"], t["l0.mix.left.k.norm"] = torch.cat([one, one]), one
    t["l0.mix.left.sink"] = torch.zeros(2, dtype=torch.bfloat16)
    t["l0.mix.left.out"], t["l0.mix.right.out"], t["l0.norm1"], t["l0.ls1"] = one * 2, zero + 0.02, one, one * 3
    return m


def far_keys_and_window_edges(device, dtype):
    """The key that the last token asks for lies near, far back, across page borders, just inside and just outside the window;
    the last token is part of the prompt or decoded alone.  The oracle must tell the two sides of the edge apart clearly."""
    filler = [i for i in range(97) if i not in (ASKS, ASKED)]
    for window in (64, 65, 100, 130):
        m = sharp_attention(window)
        eng = engine(m, device, dtype)
        g = torch.Generator().manual_seed(window)
        for back in sorted({1, 2, 63, 64, window - 2, window - 1, window, window + 1}):
            for start in (0, 3, 60, 64):
                n = start + back + 1
                t = [filler[i] for i in torch.randint(0, len(filler), (n,), generator=g).tolist()]
                t[start], t[n - 1] = ASKED, ASKS
                want = oracle.forward(t, m)
                assert_close(feed_all(eng, t, [n])[-1:], want[-1:], dtype, ("prompt", window, back, start), SHARP)
                assert_close(feed_all(eng, t, [n - 1, 1])[-1:], want[-1:], dtype, ("decoded", window, back, start), SHARP)
                if back in (window - 1, window):
                    entry = m["config"]["layers"][0]
                    left = {**entry["mixer"]["left"], "mask": {"size": window + (1 if back == window else -1)}}
                    other = {**entry, "mixer": {**entry["mixer"], "left": left}}
                    moved = oracle.forward(t, {"config": {**m["config"], "layers": [other]}, "tensors": m["tensors"]})[-1] - want[-1]
                    assert moved.std() / want[-1].std() > tolerance(dtype), "a window one token off would not be noticed"


def far_memory(device, dtype):
    """A token hundreds of positions back is still in the state: nearly nothing is forgotten, and one key stands out.  Portions end
    just before, at and after it; the state of another token in its place gives clearly other logits."""
    layers = [P(heads=1, kv_heads=1, dim=8, window=4, r_heads=1, r_dim=48, r_vdim=48, r_rot=2, base=1e9, decay=[0.9995], ff=None),
              M(heads=1, dim=48, vdim=48, cap=20.0, ff=None)]
    filler = [i for i in range(97) if i not in (ASKS, ASKED, 12)]
    for layer in (0, 1):
        m = oracle.random_model(4, layers=[layers[layer]], width=48, side_dim=4)
        t = m["tensors"]
        a, b, c = (oracle.rms_divide(t["embed"][i].float(), 1e-9) for i in (ASKS, ASKED, 12))
        basis = torch.linalg.qr(torch.stack([a, b, c]).T)[0]                 # the fillers' embeddings have no part along a, b and c
        t["embed"][filler] = (t["embed"][filler].float() @ (torch.eye(48) - basis @ basis.T)).to(torch.bfloat16)
        p = "l0.mix.right." if layer == 0 else "l0.mix."
        t[p + "q"] = (torch.outer(b, a) / 6).to(torch.bfloat16)
        t[p + "k"] = (4 * (torch.outer(b, b) + torch.outer(b, c)) / 48).to(torch.bfloat16)       # only these two tokens write along b
        if layer == 0:
            t["l0.mix.left.out"] = torch.full((48,), 0.02, dtype=torch.bfloat16)
        else:
            t["l0.mix.f.b"], t["l0.mix.f"] = torch.full((1,), 9.0, dtype=torch.bfloat16), torch.zeros(1, 48, dtype=torch.bfloat16)
        eng = engine(m, device, dtype)
        g = torch.Generator().manual_seed(layer)
        for back in (1, 63, 127, 128, 129, 400):
            ids = [filler[i] for i in torch.randint(0, len(filler), (back + 4,), generator=g).tolist()]
            ids[3], ids[-1] = ASKED, ASKS
            n, want = len(ids), oracle.forward(ids, m)
            for cuts in ([n], [n - 1, 1], [3, 1, max(1, n - 5), 1], [4, 2, n], [2, n]):
                assert_close(feed_all(eng, ids, cuts)[-1:], want[-1:], dtype, (layer, back, cuts), SHARP)
            moved = oracle.forward(ids[:3] + [12] + ids[4:], m)[-1] - want[-1]
            assert moved.std() / want[-1].std() > tolerance(dtype), "another token in the state would not be noticed"


def gates_at_their_limits(device, dtype):
    """Input gates far above and below, forget gates that drop everything or nothing: the running maximum and the floor of the
    normaliser decide."""
    for bi, bf, cap in ((12.0, 4.0, 15.0), (-12.0, 4.0, 15.0), (0.0, -12.0, 15.0), (40.0, -40.0, 20.0), (-40.0, 40.0, 8.0), (0.0, 0.0, 0.5)):
        m = model("lstm", seed=5)
        for name in list(m["tensors"]):
            if name.endswith("mix.i.b"):
                m["tensors"][name] += bi
            if name.endswith("mix.f.b"):
                m["tensors"][name] += bf
        for layer in m["config"]["layers"]:
            layer["mixer"] = {**layer["mixer"], "gate_cap": cap}
        eng, t = engine(m, device, dtype), tokens(150, 6)
        want = oracle.forward(t, m)
        for cuts in ([150], [70, 1], [2, 33]):
            assert_close(feed_all(eng, t, cuts), want, dtype, (bi, bf, cap, cuts))


def sinks_matter(device, dtype):
    """A sink that takes most of the weight, and one that takes none; the first tokens of a sequence feel it most."""
    for sink in (-30.0, 0.0, 6.0):
        m = model("edges", seed=6, sink_shift=sink)
        eng = engine(m, device, dtype)
        t = tokens(140, 8)
        want = oracle.forward(t, m)
        assert_close(feed_all(eng, t, [140]), want, dtype, sink)
        assert_close(feed_all(eng, t, [1]), want, dtype, sink)


def long_decoding(device, dtype):
    m = model("both", seed=7)
    eng = engine(m, device, dtype)
    t = tokens(600, 9)
    want = oracle.forward(t, m)
    assert_close(feed_all(eng, t, [70, 1])[::7], want[::7], dtype)


def slots_used_again(device, dtype):
    """A request's state does not leak into the next one on its slot, whether that one starts with a portion or a single token."""
    m = model("both", seed=11)
    eng = engine(m, device, dtype, max_batch=1, kv_pages=5)
    for n, cuts in ((200, [200]), (40, [1]), (150, [3, 1]), (2, [2]), (1, [1]), (90, [64, 1])):
        t = tokens(n, n + 50)
        assert_close(feed_all(eng, t, cuts), oracle.forward(t, m), dtype, (n, cuts))
    assert all_free(eng)


def greedy_generation(device, dtype):
    """Through add_request / step: batches of unequal prompts, more requests than lanes, pages used again, chunked prefill."""
    m = model("both", seed=8, gain=1.3)
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
    assert all_free(small)


def prefix_cache_reuse(device, dtype):
    """A follow-up prompt resumes from the shared pages and the snapshot of the state at a block boundary."""
    from llaminar_b200.engine.prefix_cache import PrefixCache, PrefixCacheConfig
    m = model("both", seed=9)
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
    m = model("both", seed=10)
    prompts = [tokens(60, 40), tokens(62, 41)]
    sp = SamplingParams(temperature=0.0, max_tokens=80, ignore_eos=True)
    outs = engine(m, device, dtype).generate(prompts, sp)
    eng = engine(m, device, dtype, kv_pages=5)
    got = eng.generate(prompts, sp)
    assert eng.stats["preemptions"] > 0 and all(len(o) == 80 for o in got)
    assert got == outs or dtype != torch.float32
