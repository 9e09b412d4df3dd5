"""Lagedra checkpoints: a directory with `config.json` ("architecture": "Lagedra") and safetensors files.

The reader turns the configuration's layer list into a :class:`ModelConfig` and the tensors into the names of the rest of the
package: `attn_*` for grouped attention, `lin_*` for lightning attention, `ffn_*` and `ffn_*_exps` for the feed-forwards.  A directory
that was loaded can be written to a `.gguf` file and read back: the configuration travels as one JSON string.
"""
from __future__ import annotations

from typing import Mapping

import torch

from .config import Experts, GroupedAttention, LightningAttention, ModelConfig, RopeScaling, Rotary, parallel_stack
from .weights import ModelWeights, named_weights

ARCHITECTURE = "Lagedra"


def _rotary(r: dict, size: int) -> Rotary:
    s = r.get("scaling")
    out = Rotary(int(r["dims"]), float(r["base"]), RopeScaling(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])) if s else None)
    if out.dims > size or out.dims % 2:
        raise ValueError(f"rot.dims = {out.dims} does not fit a head of {size} values")
    return out


def _mixer_from_json(kind: str, m: dict):
    heads, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    if kind == "lightning":
        decay = tuple(float(x) for x in m["decay"])
        if len(decay) != heads:
            raise ValueError(f"{len(decay)} decays for {heads} heads")
        return LightningAttention(heads, dim, vdim, decay)
    if kind != "attention":
        raise ValueError(f"unknown mixer '{kind}'")
    kv_heads, taps = int(m["kv_heads"]), int(m["conv"])
    if heads % kv_heads:
        raise ValueError(f"{heads} query heads do not share {kv_heads} key heads evenly")
    if taps < 1:
        raise ValueError(f"a convolution of {taps} taps")
    return GroupedAttention(heads, kv_heads, dim, vdim, float(m["scale"]), _rotary(m["rot"], dim), int((m.get("mask") or {}).get("size") or 0),
                            softcap=float(m.get("softcap") or 0.0), qk_norm=False, conv=taps, temperature=True, value_mix=bool(m.get("v_mix")))


def _mixer_to_json(m) -> tuple[str, dict]:
    out = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
    if isinstance(m, LightningAttention):
        return "lightning", {**out, "decay": list(m.decay)}
    s = m.rotary.scaling
    rot = {"base": m.rotary.base, "dims": m.rotary.dims, "scaling": {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow} if s else None}
    return "attention", {**out, "kv_heads": m.kv_heads, "conv": m.conv, "rot": rot, "scale": m.scale, "softcap": m.softcap or None, "v_mix": m.value_mix,
                         "mask": {"size": m.window} if m.window else None}


def _mlp_from_json(mlp: dict | None) -> int | Experts:
    if not mlp:
        return 0
    if mlp["kind"] == "dense":
        return int(mlp["ff"])
    if mlp["kind"] != "moe":
        raise ValueError(f"unknown feed-forward '{mlp['kind']}'")
    r, groups = mlp["router"], mlp["router"].get("groups") or {"count": 1, "keep": 1}
    out = Experts(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), int(groups["count"]), int(groups["keep"]), float(mlp["expert"]["limit"]), bias=False)
    if out.groups < 1 or out.n % out.groups or not 0 < out.keep <= out.groups:
        raise ValueError(f"{out.n} experts do not form {out.groups} groups of which {out.keep} stay")
    if not 0 < out.top <= out.n // out.groups * out.keep:
        raise ValueError(f"{out.top} of {out.n // out.groups * out.keep} experts cannot be chosen")
    if not out.limit > 0:
        raise ValueError(f"a limit of {out.limit} on the experts' values")
    return out


def _mlp_to_json(ff: int, e: Experts | None) -> dict | None:
    if e is not None:
        return {"kind": "moe", "expert": {"ff": e.ff, "limit": e.limit}, "router": {"experts": e.n, "top": e.top, "groups": {"count": e.groups, "keep": e.keep}}}
    return {"kind": "dense", "ff": ff} if ff else None


def config_from_json(j: dict) -> ModelConfig:
    if j.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {j.get('architecture')!r} is not {ARCHITECTURE!r}")
    mixers, ffs, mixed = [], [], None
    for i, layer in enumerate(j["layers"]):
        try:
            m = _mixer_from_json(layer["type"], layer["mixer"])
            if getattr(m, "value_mix", False):
                mixed = mixed or (m.kv_heads, m.vdim)
                if (m.kv_heads, m.vdim) != mixed:
                    raise ValueError(f"values of {m.kv_heads} heads x {m.vdim} do not mix with the first ones of {mixed[0]} x {mixed[1]}")
            mixers.append(m)
            ffs.append(_mlp_from_json(layer.get("mlp")))
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
    return parallel_stack(str(j.get("name", "lagedra")), int(j["width"]), tuple(mixers), tuple(ffs), int(j["vocab"]), int(j["max_positions"]), float(j["norm"]["eps"]))


def config_to_json(c: ModelConfig) -> dict:
    """The inverse of `config_from_json`."""
    layers = []
    for i, m in enumerate(c.mixers):
        kind, mix = _mixer_to_json(m)
        layers.append({"type": kind, "mixer": mix, "mlp": _mlp_to_json(c.ff_width(i), c.experts_of(i))})
    return {"architecture": ARCHITECTURE, "name": c.name, "layers": layers, "norm": {"eps": c.rms_eps}, "vocab": c.vocab_size, "width": c.d_model,
            "max_positions": c.learned_positions}


def tensor_names(c: ModelConfig) -> list[tuple[str, str, str, tuple[int, ...]]]:
    """(checkpoint name, package name, kind, shape) of every tensor; kinds as in `weights.named_weights`."""
    d, out = c.d_model, []

    def add(src: str, dst: str, *shape: int, kind: str = "") -> None:
        out.append((src, dst, kind or ("vec", "mat", "stack")[len(shape) - 1], shape))

    add("embed", "token_embd.weight", c.vocab_size, d)
    add("pos", "position_embd.weight", c.learned_positions, d)
    add("final.norm", "output_norm.weight", 1, kind="num")
    add("head", "output.weight", c.vocab_size, d)
    for i, m in enumerate(c.mixers):
        s, p, ff, e = f"l{i}.", f"blk.{i}.", c.ff_width(i), c.experts_of(i)
        add(s + "norm1", p + "attn_norm.weight", 1, kind="num")
        add(s + "dwa", p + "depth_average.weight", i + 2)
        if isinstance(m, LightningAttention):
            for x, n in (("q", m.dim), ("k", m.dim), ("v", m.vdim), ("g", m.vdim)):
                add(f"{s}mix.{x}", f"{p}lin_{x}.weight", m.heads * n, d)
            add(s + "mix.norm", p + "lin_norm.weight", m.heads * m.vdim)
            add(s + "mix.o", p + "lin_output.weight", d, m.heads * m.vdim)
        else:
            for x, n in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                add(f"{s}mix.{x}", f"{p}attn_{x}.weight", n, d)
                add(f"{s}mix.{x}.conv", f"{p}attn_{x}_conv.weight", n, m.conv, kind="taps")
            add(s + "mix.temp", p + "attn_temperature.weight", m.heads)
            if m.value_mix:
                add(s + "mix.vmix", p + "attn_value_mix.weight", 1, kind="num")
            add(s + "mix.o", p + "attn_output.weight", d, m.heads * m.vdim)
        if ff or e:
            add(s + "norm2", p + "ffn_norm.weight", 1, kind="num")
        if e:
            add(s + "mlp.router", p + "ffn_gate_inp.weight", e.n, d)
            add(s + "mlp.e{}.gate", p + "ffn_gate_exps.weight", e.n, e.ff, d)
            add(s + "mlp.e{}.up", p + "ffn_up_exps.weight", e.n, e.ff, d)
            add(s + "mlp.e{}.down", p + "ffn_down_exps.weight", e.n, d, e.ff)
        elif ff:
            add(s + "mlp.up", p + "ffn_up.weight", ff, d)
            add(s + "mlp.down", p + "ffn_down.weight", d, ff)
    return out


def weights_from_tensors(j: dict, tensors: Mapping[str, torch.Tensor]) -> ModelWeights:
    cfg = config_from_json(j)
    return named_weights(cfg, tensor_names(cfg), tensors)
