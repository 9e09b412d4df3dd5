"""Zogepel on the CPU back end against the plain oracle; reader, registry, command line and replay program."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from llaminar_b200.models.config import SHAPES, MatrixLSTM, ParallelMixers
from llaminar_b200.models.weights import ModelWeights
from llaminar_b200.models.zogepel import config_from_json, config_to_json, weights_from_tensors

from . import zogepel_cases as cases
from . import zogepel_oracle as oracle

F32 = torch.float32
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", cases.MODELS)
def test_whole_prompt(name):
    cases.whole_prompt(name, "cpu", F32)


@pytest.mark.parametrize("name", ["both", "parallel"])
def test_portions_and_decoding(name):
    cases.portions_and_decoding(name, "cpu", F32)


def test_token_by_token():
    cases.token_by_token("edges", "cpu", F32)


@pytest.mark.parametrize("name", ["both", "lstm"])
def test_mixed_batches(name):
    cases.mixed_batches(name, "cpu", F32)


@pytest.mark.parametrize("check", ["far_keys_and_window_edges", "far_memory", "gates_at_their_limits", "sinks_matter", "slots_used_again", "greedy_generation",
                                   "prefix_cache_reuse", "preemption"])
def test_engine(check):
    getattr(cases, check)("cpu", F32)


# -- a mistake in one mechanism is noticed (planted in the oracle) ---------------------------------------------------------------
def _scan_forgetting_at(n):
    def scan(q, k, v, *rest):
        cut = lambda x, s: x[s] if x.dim() > 1 else x                        # decays are not per token
        name = "mlstm_scan" if len(rest) == 2 else "retention_scan"
        parts = [slice(0, n), slice(n, q.shape[0])]
        return torch.cat([right[name](q[s], k[s], v[s], *(cut(x, s) for x in rest)) for s in parts])
    return scan


right = {n: getattr(oracle, n) for n in ("window_mask", "rotate", "mlstm_scan", "retention_scan", "softmax_with_sink", "mlstm_gates", "layer_norm")}


@pytest.mark.parametrize("where,wrong", [
    ("window_mask", lambda n, size: right["window_mask"](n, size + 8)), ("window_mask", lambda n, size: right["window_mask"](n, 10 ** 6)),
    ("softmax_with_sink", lambda scores, sink: torch.softmax(scores, dim=-1)),
    ("rotate", lambda x, pos, dims, base: right["rotate"](x, [p + p // 64 for p in pos], dims, base)),
    ("rotate", lambda x, pos, dims, base: x), ("mlstm_scan", _scan_forgetting_at(64)), ("retention_scan", _scan_forgetting_at(128)),
    ("mlstm_gates", lambda h, wi, bi, wf, bf, cap: right["mlstm_gates"](h, 0 * wi, bi, wf, bf, cap)),
    ("mlstm_gates", lambda h, wi, bi, wf, bf, cap: right["mlstm_gates"](h, wi, bi, wf, 0 * bf, cap)),
    ("layer_norm", lambda x, w, eps: oracle.rms_norm(x, w, eps) + 0.3), ("silu", torch.sigmoid), ("gelu_tanh", torch.relu),
    ("squared_relu", torch.relu), ("side_input", lambda x, e, T, eps: 0 * x)])
def test_a_mistake_would_be_noticed(monkeypatch, where, wrong):
    """With one mechanism wrong in the oracle the 16-bit tolerance of the engine checks is exceeded."""
    m, t = cases.model("both", seed=1), cases.tokens(230, 3)
    want = oracle.forward(t, m)
    monkeypatch.setattr(oracle, where, wrong)
    with pytest.raises(AssertionError):
        cases.assert_close(oracle.forward(t, m), want, torch.bfloat16)


# -- the oracle's own mechanisms against worked-out values ---------------------------------------------------------------------
def test_oracle_window_and_sink():
    m = oracle.window_mask(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[0].tolist() == [True] + [False] * 5
    p = oracle.softmax_with_sink(torch.zeros(1, 1, 3), torch.tensor([math.log(2.0)]))
    assert torch.allclose(p, torch.full((1, 1, 3), 0.2))


def test_oracle_rotation_keeps_relative_scores():
    q, k = torch.randn(12, dtype=torch.float64), torch.randn(12, dtype=torch.float64)
    dot = lambda i, j: oracle.rotate(q[None, None], [i], 8, 100.0)[0, 0] @ oracle.rotate(k[None, None], [j], 8, 100.0)[0, 0]
    assert torch.allclose(dot(9, 4), dot(1009, 1004))
    assert torch.equal(oracle.rotate(q[None, None], [5], 8, 100.0)[0, 0, 8:], q[8:])


def test_oracle_recurrences_written_out():
    """Both recurrences equal their unrolled sums; the mLSTM's stabiliser cancels except in the normaliser's floor."""
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(9, 2, n, generator=g, dtype=torch.float64) for n in (5, 5, 3))
    i, f = torch.randn(9, 2, generator=g, dtype=torch.float64), -torch.rand(9, 2, generator=g, dtype=torch.float64)
    for t in range(9):
        a = torch.stack([(f[j + 1:t + 1].sum(0) + i[j]).exp() for j in range(t + 1)])            # weight of token j at t, [t + 1, H]
        num = torch.einsum("jh,jhd,hd,jhe->he", a, k[:t + 1], q[t], v[:t + 1])
        den = torch.einsum("jh,jhd,hd->h", a, k[:t + 1], q[t]).abs()
        top = torch.zeros(2, dtype=torch.float64)
        for j in range(t + 1):
            top = torch.maximum(f[j] + top, i[j])
        want = num / (torch.maximum(den, torch.ones_like(den)) + 1e-6 * top.exp())[:, None]
        assert torch.allclose(oracle.mlstm_scan(q, k, v, i, f)[t], want)
        d = torch.tensor([0.5, 0.9], dtype=torch.float64)
        w = torch.stack([d ** (t - j) for j in range(t + 1)])
        assert torch.allclose(oracle.retention_scan(q, k, v, d)[t], torch.einsum("jh,jhd,hd,jhe->he", w, k[:t + 1], q[t], v[:t + 1]))


# -- configuration, files, registry --------------------------------------------------------------------------------------------
def test_config_round_trip_and_errors():
    m = cases.model("both")
    c = config_from_json(m["config"])
    assert c.has_mixers and c.has_state and not c.is_attention_stack
    assert [type(x) for x in c.mixers] == [MatrixLSTM, ParallelMixers] * 2 and c.mixers[3].left.window == 77 and c.mixers[2].gate_cap == 4.0
    assert config_from_json(config_to_json(c)) == c
    for name in cases.MODELS:
        c = config_from_json(cases.model(name)["config"])
        assert config_from_json(json.loads(json.dumps(config_to_json(c)))) == c
    change = lambda **kw: {**m["config"], **kw}
    layer = lambda **kw: change(layers=[{**m["config"]["layers"][0], **kw}])
    for bad, what in ((layer(type="other"), "mixer"), (layer(mlp={"kind": "routed"}), "feed-forward"), (change(architecture="Other"), "architecture")):
        with pytest.raises(ValueError, match=what):
            config_from_json(bad)
    for left, rt, what in (({"kv_heads": 3}, {}, "share"), ({"vdim": 5}, {}, "sizes"), ({}, {"decay": [0.5]}, "decays"), ({}, {"rot": {"base": 10.0, "dims": 22}}, "rot.dims")):
        mix = m["config"]["layers"][1]["mixer"]
        with pytest.raises(ValueError, match=what):
            config_from_json(change(layers=[{**m["config"]["layers"][1], "mixer": {"left": {**mix["left"], **left}, "right": {**mix["right"], **rt}}}]))
    t = dict(m["tensors"])
    t.pop("l1.mix.left.sink")
    with pytest.raises(KeyError, match="l1.mix.left.sink"):
        weights_from_tensors(m["config"], t)
    t["l1.mix.left.sink"] = torch.zeros(9)
    with pytest.raises(ValueError, match="shape"):
        weights_from_tensors(m["config"], t)


def test_directory_and_gguf_round_trip(tmp_path):
    m = cases.model("both")
    oracle.save(m, tmp_path / "model")
    w = ModelWeights.from_path(str(tmp_path / "model"))
    assert torch.equal(w["token_embd.weight"].to_float(), m["tensors"]["embed"].float())
    assert torch.equal(w["blk.1.ret_k.weight"].to_float(), m["tensors"]["l1.mix.right.k"].float())
    w.save_gguf(str(tmp_path / "m.gguf"))
    w2 = ModelWeights.from_path(str(tmp_path / "m.gguf"))
    assert w2.config == w.config and set(w2.tensors) == set(w.tensors)
    assert all(torch.equal(w2[n].to_float(), w[n].to_float()) for n in w.tensors)


def test_cache_and_state_layout():
    eng = cases.engine(cases.model("both"), "cpu")
    assert [tuple(l.shape[1:]) for l in eng.kv.layers] == [(2, 2, 64, 24), (2, 3, 64, 16)]
    assert eng.kv.page_bytes == (2 * 2 * 24 + 2 * 3 * 16) * 64 * 4
    st = eng.kv.hybrid
    assert [[tuple(t.shape[1:]) for t in l] for l in st.layers] == [[(3, 16, 24), (3, 24), (3,)], [(3, 28, 20)], [(2, 40, 16), (2, 16), (2,)], [(2, 16, 32)]]
    assert st.n_slots == 4 and st.slot_bytes == st.bytes_per_slot(eng.model.state_shapes)
    only = cases.engine(cases.model("lstm"), "cpu")                    # no layer with a cache: pages count tokens, hold no bytes
    assert only.kv.layers == [] and only.kv.page_bytes == 0


def test_feed_refuses_bad_steps_and_too_many_requests():
    from llaminar_b200.engine.kv_cache import OutOfPages
    eng = cases.engine(cases.model("both"), "cpu", max_context=128)
    r = eng.open_sequence()
    for tokens, want in (([], []), ([97], []), ([1], [1]), (list(range(90)) * 2, [])):
        with pytest.raises(ValueError):
            eng.feed([(r, tokens, want)])
    assert eng.feed([(r, [1, 2], [])]) is None and r.kv.length == 2
    more = [eng.open_sequence() for _ in range(3)]
    with pytest.raises(OutOfPages):
        eng.open_sequence()
    eng.close_sequence(more[0])
    eng.open_sequence()


def test_refused_combinations():
    from llaminar_b200.engine.kv_cache import Q8
    from llaminar_b200.parallel.tp_plan import TPPlan
    c = SHAPES["tiny-zogepel"]
    assert TPPlan.validate(c, 2) and not TPPlan.validate(c, 1)
    with pytest.raises(ValueError):
        cases.engine(cases.model("both"), "cpu", kv_dtype=Q8)


def test_sampled_generation_is_reproducible():
    from llaminar_b200.engine.sampling import SamplingParams
    m = cases.model("edges", gain=1.3)
    sp = SamplingParams(temperature=0.9, top_k=30, top_p=0.95, seed=5, max_tokens=10, ignore_eos=True)
    a, b = (cases.engine(m, "cpu").generate([cases.tokens(20, 1), cases.tokens(7, 2)], sp) for _ in range(2))
    assert a == b and all(len(x) == 10 for x in a)


def test_command_line(tmp_path, capsys):
    from llaminar_b200.app import main
    m = cases.model("both", gain=1.2)
    oracle.save(m, tmp_path / "model")
    argv = ["-m", str(tmp_path / "model"), "-d", "cpu", "-c", "128"]
    assert main(["oneshot", *argv, "-p", "5 9 11", "-n", "6", "--temperature", "0"]) == 0
    out = [int(x) for x in capsys.readouterr().out.split()]
    t = [5, 9, 11]
    for tok in out:
        assert tok == int(oracle.forward(t, m)[-1].argmax())
        t.append(tok)
    assert main(["plan", *argv]) == 0
    assert main(["benchmark", "--synthetic", "tiny-zogepel", "-d", "cpu", "-c", "256", "-n", "4", "--bench-prompt-tokens", "80", "--bench-runs", "1"]) == 0
    assert main(["oneshot", *argv, "-n", "2", "--kv-cache-precision", "q8_0"]) == 2


def test_memory_plan_counts_cache_and_state():
    from llaminar_b200.planning import build_plan
    c = SHAPES["zogepel-8b"]
    layout = {"pp": 1, "tp": 1, "world": 1, "stages": [("s0", ["cuda:0"], 0, -1)]}
    small, big = (build_plan(c, layout, "BF16", ctx_size=4096, batch_size=b).ranks[0] for b in (1, 9))
    pages = 4096 // 64 + 1
    per_slot = 4 * 18 * (2 * 16 * 256 * 128 + 16 * 128 + 16)
    assert big.kv_bytes - small.kv_bytes == 8 * (pages * 18 * 2 * 8 * 128 * 64 * 2 + per_slot)
    assert small.weight_bytes > 2 * 36 * 2 * 4096 * 12288


def test_trace_run_program(tmp_path):
    m = cases.model("both", seed=4)
    oracle.save(m, tmp_path / "model")
    (tmp_path / "out").mkdir()
    a, b = cases.tokens(70, 1), cases.tokens(5, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:3], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[66:67], "want": [0]}, {"id": "b", "tokens": b[3:4], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[67:], "want": [2]}], "end": ["a"]}]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", "float32", "--out", str(tmp_path / "out"),
                        "--max-tokens", "192", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    assert sorted(os.listdir(tmp_path / "out")) == ["0.f32", "2.f32", "3.f32"]
    got = lambda n: torch.frombuffer(bytearray((tmp_path / "out" / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, 97)
    wa, wb = oracle.forward(a, m), oracle.forward(b, m)
    cases.assert_close(got(0), wa[[0, 65]], F32)
    cases.assert_close(got(2), torch.stack([wa[66], wb[3]]), F32)
    cases.assert_close(got(3), wa[69:70], F32)
