"""Zogepel checkpoints: a directory with `config.json` ("architecture": "Zogepel") and safetensors files.

The reader turns the configuration's layer list into a :class:`ModelConfig` and the tensors into the package's names: `attn_*`
for windowed attention, `ret_*` for retention, `lstm_*` for the matrix LSTM, `side_*` for the per-layer token input.  A directory
that was loaded can be written to a `.gguf` file and read back: the configuration travels as one JSON string.
"""
from __future__ import annotations

from typing import Mapping

import torch

from .config import ZOGEPEL, MatrixLSTM, ModelConfig, ParallelMixers, Retention, Rotary, WindowAttention, mixer_parts
from .weights import ModelWeights, named_weights

ARCHITECTURE = "Zogepel"
CONTEXT_LENGTH = 1 << 20            # a checkpoint states no limit on positions


def _attention_from_json(m: dict) -> WindowAttention:
    heads, kv_heads, dim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    if heads % kv_heads:
        raise ValueError(f"{heads} query heads do not share {kv_heads} key heads evenly")
    if int(m.get("vdim", dim)) != dim:
        raise ValueError(f"values of {m['vdim']} are keys of {dim}: the sizes must agree")
    return WindowAttention(heads, kv_heads, dim, float(m["scale"]), int((m.get("mask") or {}).get("size") or 0))


def _retention_from_json(m: dict) -> Retention:
    out = Retention(int(m["heads"]), int(m["dim"]), int(m["vdim"]), tuple(float(x) for x in m["decay"]), Rotary(int(m["rot"]["dims"]), float(m["rot"]["base"])))
    if len(out.decay) != out.heads:
        raise ValueError(f"{len(out.decay)} decays for {out.heads} heads")
    if out.rotary.dims > out.dim or out.rotary.dims % 2:
        raise ValueError(f"rot.dims = {out.rotary.dims} does not fit a head of {out.dim} values")
    return out


def _mixer_from_json(kind: str, m: dict):
    if kind == "mlstm":
        return MatrixLSTM(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))
    if kind == "parallel":
        return ParallelMixers(_attention_from_json(m["left"]), _retention_from_json(m["right"]))
    raise ValueError(f"unknown mixer '{kind}'")


def config_from_json(j: dict) -> ModelConfig:
    if j.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {j.get('architecture')!r} is not {ARCHITECTURE!r}")
    mixers, ff = [], []
    for i, layer in enumerate(j["layers"]):
        mlp = layer.get("mlp")
        if mlp and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
        mixers.append(_mixer_from_json(layer["type"], layer["mixer"]))
        ff.append(int(mlp["ff"]) if mlp else 0)
    attn = next((m.left for m in mixers if isinstance(m, ParallelMixers)), None)
    return ModelConfig(arch="zogepel", name=str(j.get("name", "zogepel")), n_layers=len(mixers), d_model=int(j["width"]),
                       n_heads=attn.heads if attn else mixers[0].heads, n_kv_heads=attn.kv_heads if attn else 1,
                       head_dim=attn.dim if attn else mixers[0].dim, d_ff=max(ff), vocab_size=int(j["vocab"]),
                       rms_eps=float(j["norm"]["eps"]), context_length=CONTEXT_LENGTH, mixers=tuple(mixers), layer_ff=tuple(ff),
                       embed_scale=float(j["embedding"]["scale"]), residual_mult=float(j["residual_mult"]),
                       side_dim=int((j.get("token_side") or {}).get("dim") or 0), **ZOGEPEL)


def config_to_json(c: ModelConfig) -> dict:
    """The inverse of `config_from_json`."""
    layers = []
    for m, ff in zip(c.mixers, c.layer_ff):
        if isinstance(m, MatrixLSTM):
            kind, mix = "mlstm", {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
        else:
            a, r = mixer_parts(m)
            kind, mix = "parallel", {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.dim, "scale": a.scale,
                                              "mask": {"size": a.window} if a.window else None},
                                     "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay),
                                               "rot": {"base": r.rotary.base, "dims": r.rotary.dims}}}
        layers.append({"type": kind, "mixer": mix, "mlp": {"kind": "dense", "ff": ff} if ff else None})
    j = {"architecture": ARCHITECTURE, "name": c.name, "layers": layers, "norm": {"eps": c.rms_eps}, "vocab": c.vocab_size, "width": c.d_model,
         "embedding": {"scale": c.embed_scale}, "residual_mult": c.residual_mult}
    if c.side_dim:
        j["token_side"] = {"dim": c.side_dim}
    return j


def tensor_names(c: ModelConfig) -> list[tuple[str, str, str, tuple[int, ...]]]:
    """(checkpoint name, package name, kind, shape) of every tensor; kinds as in `weights.named_weights`."""
    d, v, out = c.d_model, c.vocab_size, []

    def add(src: str, dst: str, *shape: int) -> None:
        out.append((src, dst, "mat" if len(shape) == 2 else "vec", shape))

    add("embed", "token_embd.weight", v, d)
    add("final.norm", "output_norm.weight", d)
    add("head", "output.weight", v, d)
    if c.side_dim:
        add("side.embed", "side_embd.weight", v, c.side_dim * c.n_layers)
    for i, (m, ff) in enumerate(zip(c.mixers, c.layer_ff)):
        s, p = f"l{i}.", f"blk.{i}."
        add(s + "norm1", p + "post_attention_norm.weight", d)
        add(s + "ls1", p + "post_attention_scale.weight", d)
        if isinstance(m, MatrixLSTM):
            for x, n in (("q", m.dim), ("k", m.dim), ("v", m.vdim), ("g", m.vdim)):
                add(f"{s}mix.{x}", f"{p}lstm_{x}.weight", m.heads * n, d)
            add(s + "mix.o", p + "lstm_output.weight", d, m.heads * m.vdim)
            add(s + "mix.norm", p + "lstm_norm.weight", m.heads * m.vdim)
            for x in "if":
                add(f"{s}mix.{x}", f"{p}lstm_{x}.weight", m.heads, d)
                add(f"{s}mix.{x}.b", f"{p}lstm_{x}.bias", m.heads)
        else:
            a, r = mixer_parts(m)
            for x, n in (("q", a.heads), ("k", a.kv_heads), ("g", a.heads)):
                add(f"{s}mix.left.{x}", f"{p}attn_{'gate' if x == 'g' else x}.weight", n * a.dim, d)
            add(s + "mix.left.q.norm", p + "attn_q_norm.weight", a.heads * a.dim)
            add(s + "mix.left.k.norm", p + "attn_k_norm.weight", a.kv_heads * a.dim)
            add(s + "mix.left.sink", p + "attn_sinks.weight", a.heads)
            add(s + "mix.left.o", p + "attn_output.weight", d, a.heads * a.dim)
            for x, n in (("q", r.dim), ("k", r.dim), ("v", r.vdim), ("g", r.vdim)):
                add(f"{s}mix.right.{x}", f"{p}ret_{x}.weight", r.heads * n, d)
            add(s + "mix.right.o", p + "ret_output.weight", d, r.heads * r.vdim)
            add(s + "mix.left.out", p + "attn_out_norm.weight", d)
            add(s + "mix.right.out", p + "ret_out_norm.weight", d)
        if ff:
            add(s + "norm2", p + "post_ffw_norm.weight", d)
            add(s + "ls2", p + "post_ffw_scale.weight", d)
            add(s + "mlp.up", p + "ffn_up.weight", ff, d)
            add(s + "mlp.down", p + "ffn_down.weight", d, ff)
        if c.side_dim:
            add(s + "side.gate", p + "side_gate.weight", c.side_dim, d)
            add(s + "side.proj", p + "side_proj.weight", d, c.side_dim)
            add(s + "side.norm", p + "side_norm.weight", d)
    return out


def weights_from_tensors(j: dict, tensors: Mapping[str, torch.Tensor]) -> ModelWeights:
    cfg = config_from_json(j)
    return named_weights(cfg, tensor_names(cfg), tensors)
