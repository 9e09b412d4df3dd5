"""Zogepel on the GPU against the plain oracle, in bf16 and in 32-bit mode, with and without the tcgen05 prompt kernels."""
import pytest
import torch

from llaminar_b200 import ops
from llaminar_b200.engine.sampling import SamplingParams

from . import zogepel_cases as cases
from . import zogepel_oracle as oracle

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
both = pytest.mark.parametrize("dtype", [BF, F32])


@both
@pytest.mark.parametrize("name", [*cases.MODELS, "wide"])
def test_whole_prompt(name, dtype):
    cases.whole_prompt(name, "cuda", dtype)


@both
@pytest.mark.parametrize("name", ["both", "lstm", "parallel", "wide"])
def test_portions_and_decoding(name, dtype):
    cases.portions_and_decoding(name, "cuda", dtype)


@both
@pytest.mark.parametrize("name", ["edges", "wide"])
def test_token_by_token(name, dtype):
    cases.token_by_token(name, "cuda", dtype)


@both
@pytest.mark.parametrize("name", ["both", "lstm", "wide"])
def test_mixed_batches(name, dtype):
    cases.mixed_batches(name, "cuda", dtype)


@both
@pytest.mark.parametrize("check", ["far_keys_and_window_edges", "far_memory", "gates_at_their_limits", "sinks_matter", "long_decoding", "slots_used_again",
                                   "greedy_generation", "prefix_cache_reuse", "preemption"])
def test_engine(check, dtype):
    getattr(cases, check)("cuda", dtype)


@pytest.mark.parametrize("attn_tc,linear_tc", [(True, False), (False, True), (False, False)])
def test_kernel_forms_agree(attn_tc, linear_tc):
    m = cases.model("wide", seed=5)
    t = cases.tokens(430, 6)
    want = oracle.forward(t, m)
    eng = cases.engine(m, "cuda", BF)
    eng.model.stack.attn_tc, eng.model.stack.linear_tc = attn_tc, linear_tc
    cases.assert_close(cases.feed_all(eng, t, [300, 3, 90, 1]), want, BF)
    eng.check_health()


def test_long_context_many_chunks():
    """A few thousand tokens: many chunks of state, windows of several key tiles; the decode step splits the keys."""
    M, P = oracle.mlstm_layer, oracle.parallel_layer
    layers = [P(heads=4, kv_heads=1, dim=128, window=1500, r_heads=2, r_dim=64, r_vdim=64, r_rot=64, decay=[0.999, 0.98], ff=None),
              M(heads=2, dim=64, vdim=72, ff=None), P(heads=2, kv_heads=2, dim=64, window=5000, r_heads=1, r_dim=32, r_vdim=32, r_rot=16, ff=None)]
    m = oracle.random_model(3, layers=layers, width=64)
    t = cases.tokens(2100, 7)
    want = oracle.forward(t, m, dt=torch.float32)
    eng = cases.engine(m, "cuda", BF, max_context=2176, kv_pages=40, max_prefill_tokens=2176)
    for cuts in ([2085, 1], [1000, 7, 1000, 78, 1]):
        cases.assert_close(cases.feed_all(eng, t, cuts), want, BF, cuts)


@both
@pytest.mark.parametrize("width", [50, 33, 72])
def test_widths_off_the_vector_sizes(width, dtype):
    m = cases.model("edges", seed=11, width=width, vocab=101, side_dim=7)
    t = cases.tokens(150, 12)
    want = oracle.forward(t, m)
    eng = cases.engine(m, "cuda", dtype)
    for cuts in ([150], [120, 7, 1]):
        cases.assert_close(cases.feed_all(eng, t, cuts), want, dtype, cuts)


def test_sizes_without_a_tensor_core_kernel():
    """Heads beyond the attention and chunk kernels, and more query heads per key head than the decode kernel takes."""
    M, P = oracle.mlstm_layer, oracle.parallel_layer
    m = oracle.random_model(5, layers=[P(heads=2, dim=136, window=70, r_dim=200, r_rot=200, r_vdim=24), M(heads=2, dim=264, vdim=40),
                                       P(heads=34, kv_heads=2, dim=16, window=50, r_heads=1)], width=48)
    t = cases.tokens(170, 13)
    want = oracle.forward(t, m)
    eng = cases.engine(m, "cuda", BF)
    for cuts in ([170], [100, 30, 1]):
        cases.assert_close(cases.feed_all(eng, t, cuts), want, BF, cuts)


def test_captured_and_eager_decode_agree_and_launch_own_kernels():
    """In 32-bit mode both give the same tokens; in bf16 (the key splits depend on the table's width) logits within rounding."""
    m = cases.model("wide", seed=2, gain=1.3)
    prompts = [cases.tokens(n, n) for n in (5, 100, 64)]
    greedy = SamplingParams(temperature=0.0, max_tokens=20, ignore_eos=True)
    sampled = SamplingParams(temperature=0.9, top_k=30, top_p=0.95, seed=5, max_tokens=12, ignore_eos=True)
    a, b = cases.engine(m, "cuda", F32), cases.engine(m, "cuda", F32, use_graphs=False)
    n0 = ops.launch_count()
    for sp in (greedy, sampled):
        assert a.generate(prompts, sp) == b.generate(prompts, sp)
    assert a.stats["graph_replays"] > 0 and ops.launch_count() > n0
    a, b = cases.engine(m, "cuda", BF), cases.engine(m, "cuda", BF, use_graphs=False)
    t = cases.tokens(150, 3)
    cases.assert_close(cases.feed_all(a, t, [120, 1]), cases.feed_all(b, t, [120, 1]).cpu(), BF)
    assert a.stats["graph_replays"] > 0


def test_logits_do_not_depend_on_the_batch():
    """Steps of one to four sequences of different lengths: a sequence's logits stay within rounding of its own alone."""
    m = cases.model("both", seed=3)
    eng = cases.engine(m, "cuda", BF)
    t = [cases.tokens(n, n) for n in (30, 150, 64, 129)]
    alone = [cases.feed_all(eng, x, [len(x) - 4, 1]) for x in t]
    seqs = [eng.open_sequence() for _ in t]
    eng.feed([(s, x[:-4], []) for s, x in zip(seqs, t)])
    for k in range(-4, 0):
        got = eng.feed([(s, [x[k]], [0]) for s, x in zip(seqs, t)])
        cases.assert_close(got, torch.stack([a[k] for a in alone]).cpu(), BF)


def test_synthetic_shape_through_the_engine():
    from llaminar_b200.engine.engine import LLMEngine
    from llaminar_b200.models.config import SHAPES
    from llaminar_b200.models.synth import synthesize
    eng = LLMEngine(synthesize(SHAPES["tiny-zogepel"], "BF16", seed=0), device="cuda", max_batch=16, max_context=512)
    outs = eng.generate([cases.tokens(n, n, 1024) for n in (300, 7, 64, 65, 128, 20, 33, 90, 5, 6, 8, 200)], SamplingParams(temperature=0.0, max_tokens=16, ignore_eos=True))
    assert all(len(o) == 16 for o in outs)
