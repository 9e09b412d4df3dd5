"""Kefasun on the CPU back end against the plain oracle; reader, registry, command line and replay program."""
import json
import os
import subprocess
import sys

import pytest
import torch

from llaminar_b200.models.config import SHAPES, Experts, GroupedAttention, LatentAttention, Rotary
from llaminar_b200.models.kefasun import config_from_json, config_to_json, weights_from_tensors
from llaminar_b200.models.weights import ModelWeights

from . import kefasun_cases as cases
from . import kefasun_oracle as oracle
from .pozivik_oracle import save

F32 = torch.float32
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", cases.MODELS)
def test_whole_prompt(name):
    cases.whole_prompt(name, "cpu", F32)


@pytest.mark.parametrize("name", ["kinds", "order", "loop_middle", "loop_all"])
def test_portions_and_decoding(name):
    cases.portions_and_decoding(name, "cpu", F32)


def test_token_by_token():
    cases.token_by_token("loop_once", "cpu", F32)


@pytest.mark.parametrize("name", ["kinds", "order", "loop_end"])
def test_mixed_batches(name):
    cases.mixed_batches(name, "cpu", F32)


@pytest.mark.parametrize("check", cases.ENGINE_CHECKS)
def test_engine(check):
    getattr(cases, check)("cpu", F32)


right = {n: getattr(oracle, n) for n in dir(oracle) if callable(getattr(oracle, n))}


@pytest.mark.parametrize("where,wrong", [
    ("chunk_mask", lambda n, size: right["chunk_mask"](n, size + 1)), ("chunk_mask", lambda n, size: right["window_mask"](n, size)),
    ("window_mask", lambda n, size: right["window_mask"](n, size + 1)), ("window_mask", lambda n, size: right["chunk_mask"](n, size)),
    ("softmax_plus_one", lambda s: torch.softmax(s, -1)), ("softmax_with_sink", lambda s, sink: torch.softmax(s, -1)),
    ("plain_softmax", lambda s: right["softmax_plus_one"](s)), ("soft_cap", lambda s, cap: s),
    ("rotate_neighbours", lambda x, p, rot: right["rotate_halves"](x, p, rot)), ("rotate_halves", lambda x, p, rot: right["rotate_neighbours"](x, p, rot)),
    ("rotate_halves", lambda x, p, rot: right["rotate_halves"](x, [i + i // 64 for i in p], rot)),
    ("head_gate", lambda o, z: o), ("value_gate", lambda o, z: o), ("silu", lambda z: torch.nn.functional.gelu(z)),
    ("route", lambda h, T, top: (right["route"](h, T, top)[0], torch.full_like(right["route"](h, T, top)[1], 1 / top))),
    ("route", lambda h, T, top: right["route"](h, lambda n: T(n) * (n != "router.b"), top)),
    ("enter_pass", lambda x, x0, t, W: right["enter_pass"](x, x0, 0, W)), ("enter_pass", lambda x, x0, t, W: right["enter_pass"](x, x, t, W))])
def test_a_mistake_would_be_noticed(monkeypatch, where, wrong):
    """With one mechanism wrong in the oracle the 16-bit tolerance of the engine checks is exceeded."""
    m, t = cases.model("kinds", seed=1), cases.tokens(20 if where == "plain_softmax" else 230, 3)        # one in the denominator shows among few keys
    want = oracle.forward(t, m)
    monkeypatch.setattr(oracle, where, wrong)
    monkeypatch.setattr(oracle, "MIXERS", {"attention": oracle.chunked_attention, "latent_attention": oracle.latent_attention, "attention_2": oracle.capped_attention})
    with pytest.raises(AssertionError):
        cases.assert_close(oracle.forward(t, m), want, torch.bfloat16)


# -- the oracle's own mechanisms against worked-out values ---------------------------------------------------------------------
def test_oracle_masks():
    m = oracle.chunk_mask(7, 3)
    assert m[5].tolist() == [False] * 3 + [True] * 3 + [False] and m[3].tolist() == [False] * 3 + [True] + [False] * 3 and m[2].tolist() == [True] * 3 + [False] * 4
    assert oracle.window_mask(6, 3)[5].tolist() == [False] * 3 + [True] * 3 and oracle.causal_mask(4)[3].all()


def test_oracle_softmaxes():
    assert torch.allclose(oracle.softmax_plus_one(torch.zeros(1, 1, 3)), torch.full((1, 1, 3), 0.25))
    assert torch.allclose(oracle.softmax_with_sink(torch.zeros(1, 1, 3), torch.tensor([2.0]).log()), torch.full((1, 1, 3), 0.2))
    assert torch.allclose(oracle.soft_cap(torch.tensor([0.01, 1e6, -1e6]), 5.0), torch.tensor([0.01, 5.0, -5.0]), atol=1e-6)


def test_oracle_rotations():
    x, rot = torch.randn(9, 12, dtype=torch.float64), {"dims": 8, "base": 100.0}
    order = Rotary(8, 100.0, interleaved=True).halves_order(12)
    assert order == [0, 2, 4, 6, 1, 3, 5, 7, 8, 9, 10, 11]
    assert torch.allclose(oracle.rotate_neighbours(x, range(9), rot)[:, order], oracle.rotate_halves(x[:, order], range(9), rot))
    assert Rotary(8, 100.0).halves_order(12) == list(range(12))
    dot = lambda i, j: oracle.rotate_neighbours(x[0][None], [i], rot)[0] @ oracle.rotate_neighbours(x[1][None], [j], rot)[0]
    assert torch.allclose(dot(9, 4), dot(1009, 1004)) and torch.equal(oracle.rotate_neighbours(x, range(9), rot)[:, 8:], x[:, 8:])


def test_oracle_routing():
    T = lambda name: {"router": torch.eye(3), "router.b": torch.tensor([0.0, 0.0, 5.0])}[name]
    ids, w = oracle.route(torch.tensor([[3.0, 1.0, 0.0], [0.0, 9.0, 1.0]]), T, 2)
    assert ids.tolist() == [[2, 0], [1, 2]]
    assert torch.allclose(w, torch.softmax(torch.tensor([[5.0, 3.0], [9.0, 6.0]]), -1))
    assert oracle.router_gap(torch.tensor([[3.0, 1.0, 0.0]]), T, 2).item() == 2.0


# -- configuration, files, registry --------------------------------------------------------------------------------------------
def test_config_round_trip_and_errors():
    m = cases.model("kinds")
    c = config_from_json(m["config"])
    assert c.is_attention_stack and not c.has_state and [type(x) for x in c.mixers] == [GroupedAttention, LatentAttention, GroupedAttention]
    assert (c.mixers[0].chunk, c.mixers[1].window, c.mixers[2].softcap) == (20, 20, 3.0) and c.layer_ff == (0, 56, 0)
    assert c.layer_experts == (Experts(5, 2, 40), None, Experts(4, 1, 24)) and c.logit_scale == 0.7
    assert c.layer_runs() == [(0, True), (1, False), (0, True), (1, False), (2, False)]
    for name in cases.MODELS:
        c = config_from_json(cases.model(name)["config"])
        assert config_from_json(json.loads(json.dumps(config_to_json(c)))) == c
    layer = lambda i, **kw: {**m["config"], "layers": [{**m["config"]["layers"][i], **kw}]}
    mixer = lambda i, **kw: layer(i, mixer={**m["config"]["layers"][i]["mixer"], **kw})
    for bad, what in ((layer(0, type="other"), "mixer"), (layer(0, mlp={"kind": "other"}), "feed-forward"), ({**m["config"], "architecture": "Other"}, "architecture"),
                      (mixer(0, kv_heads=3), "share"), (mixer(2, rot={"base": 10.0, "dims": 18}), "rot.dims"), (mixer(1, rot={"base": 10.0, "dims": 7}), "rot.dims"),
                      (layer(0, mlp=oracle.moe(3, 4, 8)), "chosen"), ({**m["config"], "loop": {"start": 1, "stop": 5, "times": 2}}, "loop")):
        with pytest.raises(ValueError, match=what):
            config_from_json(bad)
    t = dict(m["tensors"])
    t.pop("l0.mlp.e3.up")
    with pytest.raises(KeyError, match="l0.mlp.e3.up"):
        weights_from_tensors(m["config"], t)
    t["l0.mlp.e3.up"] = torch.zeros(9, 2)
    with pytest.raises(ValueError, match="shape"):
        weights_from_tensors(m["config"], t)


def test_directory_and_gguf_round_trip(tmp_path):
    m = cases.model("loop_middle")
    save(m, tmp_path / "model")
    w = ModelWeights.from_path(str(tmp_path / "model"))
    assert torch.equal(w["token_embd.weight"].to_float(), m["tensors"]["embed"].float())
    assert torch.equal(w["blk.2.ffn_down_exps.weight"].to_float()[7], m["tensors"]["l2.mlp.e7.down"].float())
    w.save_gguf(str(tmp_path / "m.gguf"))
    w2 = ModelWeights.from_path(str(tmp_path / "m.gguf"))
    assert w2.config == w.config and set(w2.tensors) == set(w.tensors)
    assert all(torch.equal(w2[n].to_float(), w[n].to_float()) for n in w.tensors)


def test_cache_layout_per_layer_run():
    eng = cases.engine(cases.model("kinds"), "cpu")
    per_pass = [(2, 2, 64, 24), (64, 48)]
    assert [tuple(l.shape[1:]) for l in eng.kv.layers] == per_pass * 2 + [(2, 2, 64, 24)]
    assert eng.kv.page_bytes == (3 * 2 * 2 * 24 + 2 * 48) * 64 * 4 == eng.kv.bytes_per_page(0, 0, 0, 4, eng.model.kv_layer_shapes)


def test_router_statistics():
    class Stats:
        seen = []

        def record(self, layer, ids):
            self.seen.append((layer, tuple(ids.shape)))
    eng = cases.engine(cases.model("kinds"), "cpu")
    eng.model.expert_stats = Stats()
    cases.feed_all(eng, cases.tokens(9, 1), [9])
    assert Stats.seen == [(0, (9, 2)), (0, (9, 2)), (2, (9, 1))]


def test_refused_combinations():
    from llaminar_b200.engine.kv_cache import Q8
    from llaminar_b200.parallel.tp_plan import TPPlan
    c = SHAPES["tiny-kefasun"]
    assert TPPlan.validate(c, 2) and not TPPlan.validate(c, 1)
    with pytest.raises(ValueError):
        cases.engine(cases.model("kinds"), "cpu", kv_dtype=Q8)


def test_memory_plan_counts_cache_layers_and_experts():
    from llaminar_b200.planning import build_plan
    c = SHAPES["kefasun-8b"]
    layout = {"pp": 1, "tp": 1, "world": 1, "stages": [("s0", ["cuda:0"], 0, -1)]}
    small, big = (build_plan(c, layout, "BF16", ctx_size=4096, batch_size=b).ranks[0] for b in (1, 9))
    assert big.kv_bytes - small.kv_bytes == 8 * (4096 // 64 + 1) * 64 * 2 * (8 * 2 * 8 * 128 + 8 * 576)
    assert small.weight_bytes > 2 * (12 * 32 * 3 * 1536 * 4096 + 4 * 3 * 12288 * 4096)


def test_command_line(tmp_path, capsys):
    from llaminar_b200.app import main
    m = cases.model("loop_middle", gain=1.2)
    save(m, tmp_path / "model")
    argv = ["-m", str(tmp_path / "model"), "-d", "cpu", "-c", "128"]
    assert main(["oneshot", *argv, "-p", "5 9 11", "-n", "6", "--temperature", "0"]) == 0
    out = [int(x) for x in capsys.readouterr().out.split()]
    t = [5, 9, 11]
    for tok in out:
        assert tok == int(oracle.forward(t, m)[-1].argmax())
        t.append(tok)
    assert main(["plan", *argv]) == 0
    assert main(["benchmark", "--synthetic", "tiny-kefasun", "-d", "cpu", "-c", "256", "-n", "4", "--bench-prompt-tokens", "80", "--bench-runs", "1"]) == 0
    assert main(["oneshot", *argv, "-n", "2", "--kv-cache-precision", "q8_0"]) == 2


def test_trace_run_program(tmp_path):
    m = cases.model("kinds", seed=4)
    save(m, tmp_path / "model")
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
