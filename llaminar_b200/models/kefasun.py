"""Kefasun checkpoints: a directory with `config.json` ("architecture": "Kefasun") and safetensors files.

The reader turns the configuration's layer list into a :class:`ModelConfig` and the tensors into the names of the rest of the
package: GGUF names, `attn_*` for both kinds of grouped attention and for latent attention, `ffn_*_exps` for the stacked experts.  A
directory that was loaded can be written to a `.gguf` file and read back: the configuration travels as one JSON string.
"""
from __future__ import annotations

from typing import Mapping

import torch

from .config import Experts, GroupedAttention, LatentAttention, ModelConfig, Rotary, attention_stack
from .weights import ModelWeights, named_weights

ARCHITECTURE = "Kefasun"
CONTEXT_LENGTH = 1 << 20            # a checkpoint states no limit on positions


def _rotary(m: dict, size: int, interleaved: bool) -> Rotary:
    out = Rotary(int(m["rot"]["dims"]), float(m["rot"]["base"]), interleaved=interleaved)
    if out.dims > size or out.dims % 2:
        raise ValueError(f"rot.dims = {out.dims} does not fit a rotated part of {size} values")
    return out


def _mask_size(m: dict) -> int:
    return int((m.get("mask") or {}).get("size") or 0)


def _grouped(m: dict, interleaved: bool, **kw) -> GroupedAttention:
    heads, kv_heads, dim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    if heads % kv_heads:
        raise ValueError(f"{heads} query heads do not share {kv_heads} key heads evenly")
    return GroupedAttention(heads, kv_heads, dim, int(m["vdim"]), float(m["scale"]), _rotary(m, dim, interleaved), **kw)


def _mixer_from_json(kind: str, m: dict):
    if kind == "attention":
        return _grouped(m, True, chunk=_mask_size(m), null_key=True, gate="head")
    if kind == "attention_2":
        return _grouped(m, False, softcap=float(m.get("softcap") or 0.0), gate="value")
    if kind == "latent_attention":
        rot_dim = int(m["rot_dim"])
        return LatentAttention(int(m["heads"]), int(m["dim"]), rot_dim, int(m["vdim"]), int(m["q_rank"]), int(m["kv_rank"]), float(m["scale"]),
                               _rotary(m, rot_dim, True), _mask_size(m), gated=True)
    raise ValueError(f"unknown mixer '{kind}'")


def _mixer_to_json(m) -> tuple[str, dict]:
    out = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "rot": {"base": m.rotary.base, "dims": m.rotary.dims}}
    if isinstance(m, LatentAttention):
        return "latent_attention", {**out, "rot_dim": m.rot_dim, "q_rank": m.q_rank, "kv_rank": m.kv_rank, "mask": {"size": m.window} if m.window else None}
    out["kv_heads"] = m.kv_heads
    if m.gate == "head":
        return "attention", {**out, "mask": {"size": m.chunk} if m.chunk else None}
    return "attention_2", {**out, "softcap": m.softcap or None}


def _mlp_from_json(mlp: dict | None) -> int | Experts:
    if not mlp:
        return 0
    if mlp["kind"] == "dense":
        return int(mlp["ff"])
    if mlp["kind"] != "moe":
        raise ValueError(f"unknown feed-forward '{mlp['kind']}'")
    out = Experts(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]))
    if not 0 < out.top <= out.n:
        raise ValueError(f"{out.top} of {out.n} experts cannot be chosen")
    return out


def _mlp_to_json(ff: int, e: Experts | None) -> dict | None:
    if e is not None:
        return {"kind": "moe", "expert": {"ff": e.ff}, "router": {"experts": e.n, "top": e.top}}
    return {"kind": "dense", "ff": ff} if ff else None


def config_from_json(j: dict) -> ModelConfig:
    if j.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {j.get('architecture')!r} is not {ARCHITECTURE!r}")
    mixers, ffs = [], []
    for i, layer in enumerate(j["layers"]):
        try:
            mixers.append(_mixer_from_json(layer["type"], layer["mixer"]))
            ffs.append(_mlp_from_json(layer.get("mlp")))
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
    loop = j.get("loop")
    if loop:
        loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not (0 <= loop[0] < loop[1] <= len(mixers) and loop[2] >= 1):
            raise ValueError(f"loop {loop} does not fit {len(mixers)} layers")
    return attention_stack(str(j.get("name", "kefasun")), int(j["width"]), tuple(mixers), tuple(ffs), int(j["vocab"]), loop or None, float(j["norm"]["eps"]),
                           float(j["logit_scale"]), CONTEXT_LENGTH)


def config_to_json(c: ModelConfig) -> dict:
    """The inverse of `config_from_json`."""
    layers = []
    for i, m in enumerate(c.mixers):
        kind, mix = _mixer_to_json(m)
        layers.append({"type": kind, "mixer": mix, "mlp": _mlp_to_json(c.ff_width(i), c.experts_of(i))})
    j = {"architecture": ARCHITECTURE, "name": c.name, "layers": layers, "norm": {"eps": c.rms_eps}, "vocab": c.vocab_size, "width": c.d_model,
         "logit_scale": c.logit_scale}
    if c.loop:
        j["loop"] = dict(zip(("start", "stop", "times"), c.loop))
    return j


def tensor_names(c: ModelConfig) -> list[tuple[str, str, str, tuple[int, ...]]]:
    """(checkpoint name, package name, kind, shape) of every tensor; kinds as in `weights.named_weights`."""
    d, out = c.d_model, []

    def add(src: str, dst: str, *shape: int) -> None:
        out.append((src, dst, ("vec", "mat", "stack")[len(shape) - 1], shape))

    add("embed", "token_embd.weight", c.vocab_size, d)
    add("final.norm", "output_norm.weight", d)
    if c.loop:
        add("loop.in", "loop_in.weight", d, 2 * d)
        add("loop.step", "loop_step.weight", c.loop[2], d)
    for i, m in enumerate(c.mixers):
        s, p, ff, e = f"l{i}.", f"blk.{i}.", c.ff_width(i), c.experts_of(i)
        add(s + "norm1", p + "attn_norm.weight", d)
        add(s + "norm1b", p + "post_attention_norm.weight", d)
        if isinstance(m, LatentAttention):
            add(s + "mix.dq", p + "attn_q_a.weight", m.q_rank, d)
            add(s + "mix.dq.norm", p + "attn_q_a_norm.weight", m.q_rank)
            add(s + "mix.uq", p + "attn_q_b.weight", m.heads * (m.dim + m.rot_dim), m.q_rank)
            add(s + "mix.dkv", p + "attn_kv_a.weight", m.kv_rank + m.rot_dim, d)
            add(s + "mix.dkv.norm", p + "attn_kv_a_norm.weight", m.kv_rank)
            add(s + "mix.uk", p + "attn_k_b.weight", m.heads * m.dim, m.kv_rank)
            add(s + "mix.uv", p + "attn_v_b.weight", m.heads * m.vdim, m.kv_rank)
            add(s + "mix.sink", p + "attn_sinks.weight", m.heads)
            add(s + "mix.g", p + "attn_gate.weight", m.heads * m.vdim, d)
        else:
            add(s + "mix.q", p + "attn_q.weight", m.heads * m.dim, d)
            add(s + "mix.k", p + "attn_k.weight", m.kv_heads * m.dim, d)
            add(s + "mix.v", p + "attn_v.weight", m.kv_heads * m.vdim, d)
            add(s + "mix.q.norm", p + "attn_q_norm.weight", m.dim)
            add(s + "mix.k.norm", p + "attn_k_norm.weight", m.dim)
            add(s + "mix.g", p + "attn_gate.weight", m.gate_width, d)
        add(s + "mix.o", p + "attn_output.weight", d, m.heads * m.vdim)
        if ff or e:
            add(s + "norm2", p + "ffn_norm.weight", d)
            add(s + "norm2b", p + "post_ffw_norm.weight", d)
        if e:
            add(s + "mlp.router", p + "ffn_gate_inp.weight", e.n, d)
            add(s + "mlp.router.b", p + "ffn_gate_inp.bias", e.n)
            add(s + "mlp.e{}.gate", p + "ffn_gate_exps.weight", e.n, e.ff, d)
            add(s + "mlp.e{}.up", p + "ffn_up_exps.weight", e.n, e.ff, d)
            add(s + "mlp.e{}.down", p + "ffn_down_exps.weight", e.n, d, e.ff)
        elif ff:
            add(s + "mlp.gate", p + "ffn_gate.weight", ff, d)
            add(s + "mlp.up", p + "ffn_up.weight", ff, d)
            add(s + "mlp.down", p + "ffn_down.weight", d, ff)
    return out


def weights_from_tensors(j: dict, tensors: Mapping[str, torch.Tensor]) -> ModelWeights:
    cfg = config_from_json(j)
    return named_weights(cfg, tensor_names(cfg), tensors)
