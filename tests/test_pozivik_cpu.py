"""Pozivik on the CPU back end against the plain oracle; reader, registry, command line and replay program."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from llaminar_b200.models.config import SHAPES, ModelConfig, Rotary, RopeScaling
from llaminar_b200.models.pozivik import config_from_json, config_to_json, weights_from_tensors
from llaminar_b200.models.weights import ModelWeights

from . import pozivik_cases as cases
from . import pozivik_oracle as oracle

F32 = torch.float32
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", cases.MODELS)
def test_whole_prompt(name):
    cases.whole_prompt(name, "cpu", F32)


@pytest.mark.parametrize("name", ["mixed", "loop_middle", "loop_all"])
def test_portions_and_decoding(name):
    cases.portions_and_decoding(name, "cpu", F32)


def test_token_by_token():
    cases.token_by_token("loop_once", "cpu", F32)


@pytest.mark.parametrize("name", ["mixed", "loop_end"])
def test_mixed_batches(name):
    cases.mixed_batches(name, "cpu", F32)


@pytest.mark.parametrize("check", ["far_keys_and_window_edges", "sinks_matter", "long_decoding", "greedy_generation", "prefix_cache_reuse", "preemption"])
def test_engine(check):
    getattr(cases, check)("cpu", F32)


def _without_sink(scores, sink):
    return torch.softmax(scores, dim=-1)


@pytest.mark.parametrize("where,wrong", [
    ("window_mask", lambda n, size: oracle_window(n, size + 1)), ("window_mask", lambda n, size: oracle_window(n, max(1, size - 1))),
    ("window_mask", lambda n, size: oracle_window(n, None)), ("softmax_with_sink", _without_sink),
    ("rotate", lambda x, positions, rot: oracle_rotate(x, [p + p // 64 for p in positions], rot)),
    ("rotate", lambda x, positions, rot: oracle_rotate(x, positions, {**rot, "scaling": None})),
    ("centred_norm", lambda x, w, eps: oracle.plain_norm(x, w, eps)), ("gelu_tanh", lambda z: torch.nn.functional.silu(z))])
def test_a_mistake_would_be_noticed(monkeypatch, where, wrong):
    """With one mechanism wrong in the oracle the 16-bit tolerance of the engine checks is exceeded."""
    m, t = cases.model("loop_middle", seed=1), cases.tokens(230, 3)
    right = oracle.forward(t, m)
    monkeypatch.setattr(oracle, where, wrong)
    with pytest.raises(AssertionError):
        cases.assert_close(oracle.forward(t, m), right, torch.bfloat16)


oracle_window, oracle_rotate = oracle.window_mask, oracle.rotate


# -- the oracle's own mechanisms against worked-out values ---------------------------------------------------------------------
def test_oracle_window_and_sink():
    m = oracle.window_mask(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[0].tolist() == [True] + [False] * 5
    assert oracle.window_mask(4, None)[3].all()
    p = oracle.softmax_with_sink(torch.zeros(1, 1, 3), torch.tensor([math.log(2.0)]))
    assert torch.allclose(p, torch.full((1, 1, 3), 0.2))


def test_yarn_frequencies():
    r = Rotary(16, 1000.0, RopeScaling(4.0, 256, 16.0, 1.0))
    f, mag = oracle.rotation_frequencies({"dims": 16, "base": 1000.0, "scaling": {"factor": 4.0, "original": 256, "fast": 16.0, "slow": 1.0}})
    assert r.frequencies() == pytest.approx(f, rel=1e-12) and r.magnitude == pytest.approx(mag)
    plain = Rotary(16, 1000.0).frequencies()
    assert f[0] == plain[0] and f[-1] == pytest.approx(plain[-1] / 4)          # fast pairs keep, slow pairs stretch
    assert Rotary(16, 1000.0).magnitude == 1.0


def test_rotation_keeps_relative_scores():
    rot = {"dims": 8, "base": 100.0}
    q, k = torch.randn(12, dtype=torch.float64), torch.randn(12, dtype=torch.float64)
    dot = lambda i, j: oracle.rotate(q[None], [i], rot)[0] @ oracle.rotate(k[None], [j], rot)[0]
    assert torch.allclose(dot(9, 4), dot(1009, 1004))
    assert torch.equal(oracle.rotate(q[None], [5], rot)[0, 8:], q[8:])


# -- configuration, files, registry --------------------------------------------------------------------------------------------
def test_config_round_trip_and_errors():
    m = cases.model("mixed")
    c = config_from_json(m["config"])
    assert c.is_attention_stack and [x.window for x in c.mixers] == [20, 77, 64, 1000] and c.layer_ff == (56, 56, 0, 56)
    again = config_from_json(config_to_json(c))
    assert again == c
    looped = config_from_json(cases.model("loop_middle")["config"])
    assert looped.layer_runs() == [(0, False), (1, True), (1, True), (1, True), (2, False)]
    assert config_from_json(config_to_json(looped)) == looped
    bad = json.loads(json.dumps(m["config"]))
    bad["layers"][1]["type"] = "other"
    with pytest.raises(ValueError, match="mixer"):
        config_from_json(bad)
    t = dict(m["tensors"])
    t.pop("l2.mix.sink")
    with pytest.raises(KeyError, match="l2.mix.sink"):
        weights_from_tensors(m["config"], t)
    t["l2.mix.sink"] = torch.zeros(9)
    with pytest.raises(ValueError, match="shape"):
        weights_from_tensors(m["config"], t)


def test_directory_and_gguf_round_trip(tmp_path):
    m = cases.model("loop_middle")
    oracle.save(m, tmp_path / "model")
    w = ModelWeights.from_path(str(tmp_path / "model"))
    assert torch.equal(w["token_embd.weight"].to_float(), m["tensors"]["embed"].float())
    assert torch.equal(w["blk.1.attn_norm.weight"].to_float(), 1 + m["tensors"]["l1.norm1"].float())
    w.save_gguf(str(tmp_path / "m.gguf"))
    w2 = ModelWeights.from_path(str(tmp_path / "m.gguf"))
    assert w2.config == w.config and set(w2.tensors) == set(w.tensors)
    assert all(torch.equal(w2[n].to_float(), w[n].to_float()) for n in w.tensors)
    (tmp_path / "model" / "config.json").write_text(json.dumps({"architecture": "Unknown"}))
    with pytest.raises(ValueError, match="Unknown"):
        ModelWeights.from_path(str(tmp_path / "model"))


def test_cache_layout_per_layer_run():
    eng = cases.engine(cases.model("loop_all"), "cpu")
    assert [tuple(l.shape[1:]) for l in eng.kv.layers] == [(64, 48), (64, 48)] * 2 or len(eng.kv.layers) == 4
    assert [(l.shape[2],) for l in eng.kv.layers] == eng.model.kv_layer_shapes
    assert eng.kv.page_bytes == sum(w for w, in eng.model.kv_layer_shapes) * 64 * 4


def test_feed_refuses_bad_steps():
    eng = cases.engine(cases.model("mixed"), "cpu", max_context=128)
    r = eng.open_sequence()
    for tokens, want in (([], []), ([97], []), ([1], [1]), (list(range(90)) * 2, [])):
        with pytest.raises(ValueError):
            eng.feed([(r, tokens, want)])
    assert eng.feed([(r, [1, 2], [])]) is None and r.kv.length == 2


def test_refused_combinations():
    from llaminar_b200.engine.kv_cache import Q8
    from llaminar_b200.parallel.tp_plan import TPPlan
    c = SHAPES["tiny-pozivik"]
    assert TPPlan.validate(c, 2) and not TPPlan.validate(c, 1)
    with pytest.raises(ValueError):
        cases.engine(cases.model("mixed"), "cpu", kv_dtype=Q8)


def test_command_line(tmp_path, capsys):
    from llaminar_b200.app import main
    m = cases.model("loop_middle", gain=1.2)
    oracle.save(m, tmp_path / "model")
    argv = ["-m", str(tmp_path / "model"), "-d", "cpu", "-c", "128"]
    assert main(["oneshot", *argv, "-p", "5 9 11", "-n", "6", "--temperature", "0"]) == 0
    out = [int(x) for x in capsys.readouterr().out.split()]
    t = [5, 9, 11]
    for tok in out:
        assert tok == int(oracle.forward(t, m)[-1].argmax())
        t.append(tok)
    assert main(["plan", *argv]) == 0
    assert main(["benchmark", "--synthetic", "tiny-pozivik", "-d", "cpu", "-c", "256", "-n", "4", "--bench-prompt-tokens", "80", "--bench-runs", "1"]) == 0
    assert main(["oneshot", *argv, "-n", "2", "--kv-cache-precision", "q8_0"]) == 2


def test_trace_run_program(tmp_path):
    m = cases.model("mixed", seed=4)
    oracle.save(m, tmp_path / "model")
    (tmp_path / "out").mkdir()
    a, b = cases.tokens(70, 1), cases.tokens(5, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:3], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[66:67], "want": [0]}, {"id": "b", "tokens": b[3:4], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[67:], "want": [2]}], "end": ["a"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", "float32", "--out", str(tmp_path / "out"),
                        "--max-tokens", "192", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    assert sorted(os.listdir(tmp_path / "out")) == ["0.f32", "2.f32", "3.f32"]
    got = lambda n: torch.frombuffer(bytearray((tmp_path / "out" / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, 97)
    wa, wb = oracle.forward(a, m), oracle.forward(b, m)
    cases.assert_close(got(0), wa[[0, 65]], F32)
    cases.assert_close(got(2), torch.stack([wa[66], wb[3]]), F32)
    cases.assert_close(got(3), wa[69:70], F32)
