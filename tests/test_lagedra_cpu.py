"""Lagedra on the CPU back end against the plain oracle; reader, registry, command line and replay program."""
import json
import os
import subprocess
import sys

import pytest
import torch

from llaminar_b200.models.config import SHAPES, Experts, GroupedAttention, LightningAttention, RopeScaling, Rotary
from llaminar_b200.models.lagedra import config_from_json, config_to_json, weights_from_tensors
from llaminar_b200.models.weights import ModelWeights

from . import lagedra_cases as cases
from . import lagedra_oracle as oracle
from .pozivik_oracle import save

F32 = torch.float32
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", cases.MODELS)
def test_whole_prompt(name):
    cases.whole_prompt(name, "cpu", F32)


@pytest.mark.parametrize("name", ["kinds", "order", "pauses", "recurrent"])
def test_portions_and_decoding(name):
    cases.portions_and_decoding(name, "cpu", F32)


def test_token_by_token():
    cases.token_by_token("attending", "cpu", F32)


@pytest.mark.parametrize("name", ["kinds", "order"])
def test_mixed_batches(name):
    cases.mixed_batches(name, "cpu", F32)


@pytest.mark.parametrize("check", cases.ENGINE_CHECKS)
def test_engine(check):
    getattr(cases, check)("cpu", F32)


right = {n: getattr(oracle, n) for n in dir(oracle) if callable(getattr(oracle, n))}


def _restart(f, u, *a):
    """A function of rows that forgets what was before row 128."""
    return torch.cat([f(u[:128], *a), f(u[128:], *a)])


@pytest.mark.parametrize("where,wrong", [
    ("window_mask", lambda n, size: right["window_mask"](n, size + 1)), ("window_mask", lambda n, size: right["window_mask"](n, size - 1)),
    ("window_mask", lambda n, size: right["window_mask"](n, None)), ("head_temperature", lambda s, t: s), ("soft_cap", lambda s, cap: s),
    ("yarn", lambda rot: (right["yarn"]({**rot, "scaling": None})[0], right["yarn"](rot)[1])), ("yarn", lambda rot: (right["yarn"](rot)[0], 1.0)),
    ("rotate_halves", lambda x, p, rot: right["rotate_halves"](x, [i + i // 64 for i in p], rot)),
    ("owner", lambda h, g: [i % g for i in range(h)]),
    ("mix_values", lambda v, first, share: v), ("mix_values", lambda v, first, share: right["mix_values"](v, None if first is None else first.roll(1, 0), share)),
    ("mix_values", lambda v, first, share: right["mix_values"](v, first, 1 - share)),
    ("short_conv", lambda u, w: u), ("short_conv", lambda u, w: right["short_conv"](u, w.flip(1))), ("short_conv", lambda u, w: _restart(right["short_conv"], u, w)),
    ("decayed_state", lambda q, k, v, d: right["decayed_state"](q, k, v, d.flip(0))), ("decayed_state", lambda q, k, v, d: right["decayed_state"](q, k, v, torch.ones_like(d))),
    ("decayed_state", lambda q, k, v, d: torch.cat([right["decayed_state"](q[:128], k[:128], v[:128], d), right["decayed_state"](q[128:], k[128:], v[128:], d)])),
    ("output_gate", lambda o, z: o), ("gain_norm", lambda x, w, eps: x * w), ("gain_norm", lambda x, w, eps: right["gain_norm"](x, torch.ones_like(w), eps)),
    ("silu", lambda z: z), ("gelu_tanh", lambda z: z.relu()), ("scalar_norm", lambda x, g, eps: right["scalar_norm"](x, 1.0, eps)),
    ("add_positions", lambda x, table: x), ("add_positions", lambda x, table: x + table[1:x.shape[0] + 1]),
    ("limited_ffn", lambda h, T, limit: right["limited_ffn"](h, T, 100.0)), ("limited_ffn", lambda h, T, limit: right["silu"](h @ T("gate").T) * (h @ T("up").T) @ T("down").T),
    ("allowed_experts", lambda s, groups: torch.ones_like(s, dtype=torch.bool)), ("expert_weights", lambda s, ids: s.gather(1, ids)),
    ("depth_average", lambda xs, w: xs[-1]), ("depth_average", lambda xs, w: right["depth_average"](xs[::-1], w))])
def test_a_mistake_would_be_noticed(monkeypatch, where, wrong):
    """With one mechanism wrong in the oracle the 16-bit tolerance of the engine checks is exceeded."""
    m, t = cases.model("kinds", seed=1), cases.tokens(230, 3)
    want = oracle.forward(t, m)
    monkeypatch.setattr(oracle, where, wrong)
    got = oracle.forward(t, m)
    with pytest.raises(AssertionError):
        cases.assert_close(got, want, torch.bfloat16)


# -- the oracle's own mechanisms against worked-out values ---------------------------------------------------------------------
def test_oracle_masks_and_caps():
    m = oracle.window_mask(6, 3)
    assert m[5].tolist() == [False] * 3 + [True] * 3 and m[1].tolist() == [True, True] + [False] * 4 and oracle.window_mask(4, None)[3].all()
    assert torch.allclose(oracle.soft_cap(torch.tensor([0.01, 1e6, -1e6]), 5.0), torch.tensor([0.01, 5.0, -5.0]), atol=1e-6)


def test_oracle_conv_and_state():
    u = torch.tensor([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0]])
    w = torch.tensor([[100.0, 10.0, 1.0], [0.0, 0.0, 2.0]])
    assert oracle.short_conv(u, w).tolist() == [[1.0, 20.0], [12.0, 40.0], [123.0, 60.0]]
    q, k, v = torch.ones(3, 1, 1), torch.ones(3, 1, 1), torch.tensor([1.0, 2.0, 4.0]).view(3, 1, 1)
    assert oracle.decayed_state(q, k, v, torch.tensor([0.5])).flatten().tolist() == [1.0, 2.5, 5.25]


def test_oracle_yarn():
    rot = {"dims": 16, "base": 100.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    plain, (freqs, grow) = oracle.yarn({**rot, "scaling": None})[0], oracle.yarn(rot)
    assert freqs[0] == plain[0] and abs(freqs[-1] - plain[-1] / 4) < 1e-12 and abs(grow - 1.1386294) < 1e-6
    assert all(f / 4 - 1e-12 <= g <= f + 1e-12 for f, g in zip(plain, freqs))
    ours = Rotary(16, 100.0, RopeScaling(4.0, 64, 8.0, 1.0))
    assert torch.allclose(torch.tensor(ours.frequencies()), torch.tensor(freqs)) and abs(ours.magnitude - grow) < 1e-12


def test_oracle_routing():
    T = lambda name: torch.eye(6)
    x = torch.tensor([[5.0, 0.0, 4.0, 3.0, 1.0, 4.5]])
    ids, w = oracle.route(x, T, {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}})       # best scores of the groups: 5, 4, 4.5
    assert ids.tolist() == [[0, 5, 4]] and torch.allclose(w, torch.softmax(torch.tensor([[5.0, 4.5, 1.0]]), -1))
    ids, _ = oracle.route(x, T, {"experts": 6, "top": 3})
    assert ids.tolist() == [[0, 5, 2]]
    assert abs(oracle.router_gap(x, T, {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}}).item() - 0.5) < 1e-6


def test_oracle_limited_pairs():
    T = lambda name: {"gate": torch.tensor([[9.0]]), "up": torch.tensor([[-9.0]]), "down": torch.tensor([[1.0]])}[name]
    want = 2.0 / (1 + torch.exp(torch.tensor(-3.404))) * (-2.0 + 1.0)
    assert torch.allclose(oracle.limited_ffn(torch.ones(1, 1), T, 2.0), want)


# -- configuration, files, registry --------------------------------------------------------------------------------------------
def test_config_round_trip_and_errors():
    m = cases.model("kinds")
    c = config_from_json(m["config"])
    assert c.is_attention_stack and c.has_state and c.parallel_ff and [type(x) for x in c.mixers] == [LightningAttention, GroupedAttention, GroupedAttention, LightningAttention]
    assert (c.mixers[1].window, c.mixers[1].softcap, c.mixers[1].conv, c.mixers[2].conv) == (20, 6.0, 4, 3) and c.layer_ff == (56, 0, 72, 0)
    assert c.layer_experts == (None, Experts(6, 2, 40, 2, 1, 1.5, False), None, Experts(8, 3, 24, 4, 2, 0.8, False)) and c.context_length == 700
    for name in cases.MODELS:
        c = config_from_json(cases.model(name)["config"])
        assert config_from_json(json.loads(json.dumps(config_to_json(c)))) == c
    layer = lambda i, **kw: {**m["config"], "layers": [{**m["config"]["layers"][i], **kw}]}
    mixer = lambda i, **kw: layer(i, mixer={**m["config"]["layers"][i]["mixer"], **kw})
    other = {**m["config"], "layers": [m["config"]["layers"][1], {**m["config"]["layers"][2], "mixer": {**m["config"]["layers"][2]["mixer"], "vdim": 20}}]}
    for bad, what in ((layer(0, type="other"), "mixer"), (layer(0, mlp={"kind": "other"}), "feed-forward"), ({**m["config"], "architecture": "Other"}, "architecture"),
                      (mixer(1, kv_heads=3), "share"), (mixer(1, rot={"base": 10.0, "dims": 26}), "rot.dims"), (mixer(1, rot={"base": 10.0, "dims": 7}), "rot.dims"),
                      (mixer(0, decay=[0.5]), "decays"), (mixer(1, conv=0), "taps"), (other, "mix"), (layer(0, mlp=oracle.moe(6, 5, 8, 3, 2)), "chosen"),
                      (layer(0, mlp=oracle.moe(6, 2, 8, 4, 2)), "groups"), (layer(0, mlp=oracle.moe(6, 2, 8, 3, 4)), "groups"), (layer(0, mlp=oracle.moe(limit=0.0)), "limit")):
        with pytest.raises(ValueError, match=what):
            config_from_json(bad)
    t = dict(m["tensors"])
    t.pop("l1.mlp.e3.up")
    with pytest.raises(KeyError, match="l1.mlp.e3.up"):
        weights_from_tensors(m["config"], t)
    t["l1.mlp.e3.up"] = torch.zeros(9, 2)
    with pytest.raises(ValueError, match="shape"):
        weights_from_tensors(m["config"], t)


def test_directory_and_gguf_round_trip(tmp_path):
    from llaminar_b200.models.convert_hf import requantize
    m = cases.model("kinds")
    save(m, tmp_path / "model")
    w = ModelWeights.from_path(str(tmp_path / "model"))
    assert torch.equal(w["token_embd.weight"].to_float(), m["tensors"]["embed"].float())
    assert torch.equal(w["blk.1.attn_q_conv.weight"].to_float(), m["tensors"]["l1.mix.q.conv"].float())
    assert torch.equal(w["blk.3.ffn_down_exps.weight"].to_float()[7], m["tensors"]["l3.mlp.e7.down"].float())
    w.save_gguf(str(tmp_path / "m.gguf"))
    w2 = ModelWeights.from_path(str(tmp_path / "m.gguf"))
    assert w2.config == w.config and set(w2.tensors) == set(w.tensors)
    assert all(torch.equal(w2[n].to_float(), w[n].to_float()) for n in w.tensors)
    assert torch.equal(requantize(w, "Q8_0")["blk.1.attn_q_conv.weight"].to_float(), w["blk.1.attn_q_conv.weight"].to_float())


def test_cache_and_state_layout():
    eng = cases.engine(cases.model("kinds"), "cpu")
    assert [tuple(l.shape[1:]) for l in eng.kv.layers] == [(2, 2, 64, 24)] * 2
    assert [tuple(t.shape[1:]) for layer in eng.kv.hybrid.layers for t in layer] == [(3, 16, 24), (4, 8 * 24), (3, 8 * 24), (2, 40, 16)]
    assert cases.engine(cases.model("recurrent"), "cpu").kv.layers == []


def test_router_statistics():
    class Stats:
        seen = []

        def record(self, layer, ids):
            self.seen.append((layer, tuple(ids.shape)))
    eng = cases.engine(cases.model("kinds"), "cpu")
    eng.model.expert_stats = Stats()
    cases.feed_all(eng, cases.tokens(9, 1), [9])
    assert Stats.seen == [(1, (9, 2)), (3, (9, 3))]


def test_refused_combinations():
    from llaminar_b200.engine.kv_cache import Q8
    from llaminar_b200.parallel.tp_plan import TPPlan
    c = SHAPES["tiny-lagedra"]
    assert TPPlan.validate(c, 2) and not TPPlan.validate(c, 1)
    with pytest.raises(ValueError):
        cases.engine(cases.model("kinds"), "cpu", kv_dtype=Q8)


def test_memory_plan_counts_cache_state_and_streams():
    from llaminar_b200.planning import build_plan
    c = SHAPES["lagedra-8b"]
    layout = {"pp": 1, "tp": 1, "world": 1, "stages": [("s0", ["cuda:0"], 0, -1)]}
    small, big = (build_plan(c, layout, "BF16", ctx_size=4096, batch_size=b).ranks[0] for b in (1, 9))
    assert big.kv_bytes - small.kv_bytes == 8 * ((4096 // 64 + 1) * 64 * 2 * 8 * 2 * 8 * 128 + 4 * (8 * 16 * 128 * 256 + 8 * 4 * 48 * 128))
    assert small.weight_bytes > 2 * (8 * 32 * 3 * 1536 * 4096 + 8 * 2 * 12288 * 4096)
    assert small.activation_bytes > 8192 * 4096 * 4 * 17


def test_command_line(tmp_path, capsys):
    from llaminar_b200.app import main
    m = cases.model("kinds", gain=1.2)
    save(m, tmp_path / "model")
    argv = ["-m", str(tmp_path / "model"), "-d", "cpu", "-c", "128"]
    assert main(["oneshot", *argv, "-p", "5 9 11", "-n", "6", "--temperature", "0"]) == 0
    out = [int(x) for x in capsys.readouterr().out.split()]
    t = [5, 9, 11]
    for tok in out:
        assert tok == int(oracle.forward(t, m)[-1].argmax())
        t.append(tok)
    assert main(["plan", *argv]) == 0
    assert main(["benchmark", "--synthetic", "tiny-lagedra", "-d", "cpu", "-c", "256", "-n", "4", "--bench-prompt-tokens", "80", "--bench-runs", "1"]) == 0
    assert main(["oneshot", *argv, "-n", "2", "--kv-cache-precision", "q8_0"]) == 2
    assert main(["oneshot", "-m", str(tmp_path / "model"), "-d", "cpu", "-c", "701", "-p", "5", "-n", "2"]) == 2


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
