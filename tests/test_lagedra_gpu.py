"""Lagedra on the GPU against the plain oracle, in bf16 and in 32-bit mode, with and without the tcgen05 kernels."""
import pytest
import torch

from llaminar_b200 import ops
from llaminar_b200.engine.sampling import SamplingParams

from . import lagedra_cases as cases
from . import lagedra_oracle as oracle

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
both = pytest.mark.parametrize("dtype", [BF, F32])


@both
@pytest.mark.parametrize("name", [*cases.MODELS, "wide"])
def test_whole_prompt(name, dtype):
    cases.whole_prompt(name, "cuda", dtype)


@both
@pytest.mark.parametrize("name", ["kinds", "order", "pauses", "wide"])
def test_portions_and_decoding(name, dtype):
    cases.portions_and_decoding(name, "cuda", dtype)


@both
@pytest.mark.parametrize("name", ["attending", "recurrent", "order", "wide"])
def test_token_by_token(name, dtype):
    cases.token_by_token(name, "cuda", dtype)


@both
@pytest.mark.parametrize("name", ["kinds", "order", "wide"])
def test_mixed_batches(name, dtype):
    cases.mixed_batches(name, "cuda", dtype)


@both
@pytest.mark.parametrize("check", cases.ENGINE_CHECKS)
def test_engine(check, dtype):
    getattr(cases, check)("cuda", dtype)


@pytest.mark.parametrize("off", ["linear_tc", "prefill_tc", "fast"])
def test_kernel_forms_agree(off):
    """The forms without tcgen05, and the experts in float arithmetic."""
    m = cases.model("wide", seed=5)
    t = cases.tokens(430, 6)
    eng = cases.engine(m, "cuda", BF)
    if off == "fast":
        for L in eng.model.layers:
            if L.experts:
                L.experts.fast = False
    else:
        setattr(eng.model.stack, off, False)
    cases.assert_close(cases.feed_all(eng, t, [300, 3, 90, 1]), cases.expected(t, m), BF)
    eng.check_health()


@pytest.mark.parametrize("few,many", [(0, 1 << 30), (1 << 30, 0)])
def test_sublayers_one_after_the_other_or_at_the_same_time(few, many):
    """Both orders, in prompts, portions and captured decode steps, twice with the same result."""
    m = cases.model("wide", seed=8)
    want, t = None, cases.tokens(330, 3)
    eng = cases.engine(m, "cuda", BF)
    st = eng.model.stack
    st.beside_few, st.beside_few_experts, st.beside_many = few, few, many
    for _ in range(2):
        got = cases.feed_all(eng, t, [200, 5, 64, 1])
        cases.assert_close(got, cases.expected(t, m), BF)
        assert want is None or torch.equal(got, want)
        want = got


def test_long_context_many_tiles():
    """Windows of several key tiles and none at all, many chunks of the recurrence, over a few thousand tokens."""
    A, L = oracle.attention_entry, oracle.lightning_entry
    layers = [L(heads=2, dim=128, vdim=128, decay=(0.99, 0.9995), mlp=None), A(heads=4, kv_heads=1, dim=128, vdim=128, rot_dims=128, window=700, mlp=oracle.moe(8, 2, 64)),
              A(heads=4, kv_heads=2, dim=64, vdim=64, rot_dims=64, window=None, conv=3, v_mix=False, mlp=None)]
    m = oracle.random_model(layers, 3, width=64, max_positions=2100)
    t = cases.tokens(2100, 7)
    want = cases.expected(t, m, dt=F32)
    eng = cases.engine(m, "cuda", BF, max_context=2176, kv_pages=40, max_prefill_tokens=2176)
    for cuts in ([2085, 1], [1000, 7, 1000, 78, 1]):
        cases.assert_close(cases.feed_all(eng, t, cuts), want, BF, cuts)


@both
@pytest.mark.parametrize("width", [50, 33, 72])
def test_widths_off_the_vector_sizes(width, dtype):
    m = cases.model("kinds", seed=11, width=width, vocab=101)
    t = cases.tokens(150, 12)
    want = cases.expected(t, m)
    eng = cases.engine(m, "cuda", dtype)
    for cuts in ([150], [120, 7, 1]):
        cases.assert_close(cases.feed_all(eng, t, cuts), want, dtype, cuts)


def test_sizes_without_a_tensor_core_kernel():
    """Heads beyond the attention and chunk kernels, many query heads per key head, a filter of many taps."""
    A, L = oracle.attention_entry, oracle.lightning_entry
    m = oracle.random_model([A(heads=2, kv_heads=1, dim=200, vdim=136, window=50, conv=4, v_mix=False), L(heads=2, dim=200, vdim=72), A(heads=34, kv_heads=2, dim=16, vdim=16, conv=9)], 5)
    t = cases.tokens(170, 13)
    want = cases.expected(t, m)
    eng = cases.engine(m, "cuda", BF)
    for cuts in ([170], [100, 30, 1]):
        cases.assert_close(cases.feed_all(eng, t, cuts), want, BF, cuts)


def test_captured_and_eager_decode_agree_and_launch_own_kernels():
    m = cases.model("wide", seed=2, gain=1.3)
    prompts = [cases.tokens(n, n) for n in (5, 100, 64)]
    sp = SamplingParams(temperature=0.0, max_tokens=20, ignore_eos=True)
    a, b = cases.engine(m, "cuda", BF), cases.engine(m, "cuda", BF, use_graphs=False)
    n0 = ops.launch_count()
    assert a.generate(prompts, sp) == b.generate(prompts, sp)
    assert a.stats["graph_replays"] > 0 and ops.launch_count() > n0
    sampled = SamplingParams(temperature=0.9, top_k=30, top_p=0.95, seed=5, max_tokens=12, ignore_eos=True)
    for eng in (a, b):                                                              # the same draws every time
        assert eng.generate(prompts, sampled) == eng.generate(prompts, sampled)


def test_logits_do_not_depend_on_the_batch():
    """Steps of one to four sequences of different lengths: a sequence's logits stay within rounding of its own alone."""
    m = cases.model("kinds", seed=3)
    eng = cases.engine(m, "cuda", BF)
    t = [cases.tokens(n, n) for n in (30, 150, 64, 129)]
    alone = [cases.feed_all(eng, x, [len(x) - 4, 1]) for x in t]
    gaps = [cases.expected(x, m)[1] for x in t]
    seqs = [eng.open_sequence() for _ in t]
    eng.feed([(s, x[:-4], []) for s, x in zip(seqs, t)])
    for k in range(-4, 0):
        got = eng.feed([(s, [x[k]], [0]) for s, x in zip(seqs, t)])
        cases.assert_close(got, (torch.stack([a[k] for a in alone]).cpu(), torch.stack([g[k] for g in gaps])), BF)


def test_synthetic_shape_through_the_engine():
    from llaminar_b200.engine.engine import LLMEngine
    from llaminar_b200.models.config import SHAPES
    from llaminar_b200.models.synth import synthesize
    eng = LLMEngine(synthesize(SHAPES["tiny-lagedra"], "BF16", seed=0), device="cuda", max_batch=16, max_context=512)
    outs = eng.generate([cases.tokens(n, n, 1024) for n in (300, 7, 64, 65, 128, 20, 33, 90, 5, 6, 77)], SamplingParams(temperature=0.0, max_tokens=16, ignore_eos=True))
    assert all(len(o) == 16 for o in outs)
