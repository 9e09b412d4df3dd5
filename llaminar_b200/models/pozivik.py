"""Pozivik checkpoints: a directory with `config.json` ("architecture": "Pozivik") and safetensors files.

The reader turns the configuration's layer list into a :class:`ModelConfig` and the tensors into the names and conventions of
the rest of the package: GGUF names (the low-rank projections as `attn_q_a` / `attn_q_b`, `attn_kv_a` / `attn_k_b` /
`attn_v_b`), and norm gains as they multiply (the checkpoint's zero-centred gains become 1 + w).  A directory that was loaded
can be written to a `.gguf` file and read back: the configuration travels as one JSON string.
"""
from __future__ import annotations

from typing import Mapping

import torch

from .config import LatentAttention, ModelConfig, Rotary, RopeScaling
from .weights import ModelWeights, named_weights

ARCHITECTURE = "Pozivik"
CONTEXT_LENGTH = 1 << 20            # a checkpoint states no limit on positions


def _mixer_from_json(m: dict) -> LatentAttention:
    rot, sc = m["rot"], m["rot"].get("scaling")
    scaling = RopeScaling(float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"])) if sc else None
    mask = m.get("mask") or {}
    out = LatentAttention(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                          q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                          rotary=Rotary(int(rot["dims"]), float(rot["base"]), scaling), window=int(mask.get("size") or 0))
    if out.rotary.dims > out.rot_dim or out.rotary.dims % 2:
        raise ValueError(f"rot.dims = {out.rotary.dims} does not fit a rotated part of {out.rot_dim} values")
    return out


def config_from_json(j: dict) -> ModelConfig:
    if j.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {j.get('architecture')!r} is not {ARCHITECTURE!r}")
    mixers, ff = [], []
    for i, layer in enumerate(j["layers"]):
        if layer["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer '{layer['type']}'")
        mlp = layer.get("mlp")
        if mlp and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
        mixers.append(_mixer_from_json(layer["mixer"]))
        ff.append(int(mlp["ff"]) if mlp else 0)
    loop = j.get("loop")
    if loop:
        loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not (0 <= loop[0] < loop[1] <= len(mixers) and loop[2] >= 1):
            raise ValueError(f"loop {loop} does not fit {len(mixers)} layers")
    first = mixers[0]
    return ModelConfig(arch="pozivik", name=str(j.get("name", "pozivik")), n_layers=len(mixers), d_model=int(j["width"]),
                       n_heads=first.heads, n_kv_heads=1, head_dim=first.cache_width, d_ff=max(ff), vocab_size=int(j["vocab"]),
                       rope_theta=first.rotary.base, rms_eps=float(j["norm"]["eps"]), context_length=CONTEXT_LENGTH, qk_norm=False,
                       tie_embeddings=False, mixers=tuple(mixers), layer_ff=tuple(ff), loop=loop or None, embed_norm=True,
                       post_norms=True, ffn_act="gelu_tanh")


def config_to_json(c: ModelConfig) -> dict:
    """The inverse of `config_from_json`."""
    layers = []
    for m, ff in zip(c.mixers, c.layer_ff):
        r, s = m.rotary, m.rotary.scaling
        rot = {"base": r.base, "dims": r.dims}
        if s:
            rot["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
        layers.append({"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
                       "mixer": {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank,
                                 "kv_rank": m.kv_rank, "scale": m.scale, "rot": rot, "mask": {"size": m.window} if m.window else None}})
    j = {"architecture": ARCHITECTURE, "name": c.name, "layers": layers, "norm": {"eps": c.rms_eps}, "vocab": c.vocab_size,
         "width": c.d_model}
    if c.loop:
        j["loop"] = dict(zip(("start", "stop", "times"), c.loop))
    return j


def tensor_names(c: ModelConfig) -> list[tuple[str, str, str, tuple[int, ...]]]:
    """(checkpoint name, package name, kind, shape) of every tensor: kind "mat" a matrix, "vec" a vector kept as it is,
    "gain" a zero-centred norm gain."""
    d, v = c.d_model, c.vocab_size
    out = [("embed", "token_embd.weight", "mat", (v, d)), ("embed.norm", "token_embd_norm.weight", "gain", (d,)),
           ("final.norm", "output_norm.weight", "gain", (d,)), ("head", "output.weight", "mat", (v, d))]
    if c.loop:
        out.append(("loop.in", "loop_in.weight", "mat", (d, 2 * d)))
    for i, (m, ff) in enumerate(zip(c.mixers, c.layer_ff)):
        s, p = f"l{i}.", f"blk.{i}."
        out += [(s + "norm1", p + "attn_norm.weight", "gain", (d,)), (s + "norm1b", p + "post_attention_norm.weight", "gain", (d,)),
                (s + "mix.dq", p + "attn_q_a.weight", "mat", (m.q_rank, d)), (s + "mix.dq.norm", p + "attn_q_a_norm.weight", "vec", (m.q_rank,)),
                (s + "mix.uq", p + "attn_q_b.weight", "mat", (m.heads * (m.dim + m.rot_dim), m.q_rank)),
                (s + "mix.dkv", p + "attn_kv_a.weight", "mat", (m.kv_rank + m.rot_dim, d)),
                (s + "mix.dkv.norm", p + "attn_kv_a_norm.weight", "vec", (m.kv_rank,)),
                (s + "mix.uk", p + "attn_k_b.weight", "mat", (m.heads * m.dim, m.kv_rank)),
                (s + "mix.uv", p + "attn_v_b.weight", "mat", (m.heads * m.vdim, m.kv_rank)),
                (s + "mix.sink", p + "attn_sinks.weight", "vec", (m.heads,)),
                (s + "mix.o", p + "attn_output.weight", "mat", (d, m.heads * m.vdim))]
        if ff:
            out += [(s + "norm2", p + "ffn_norm.weight", "gain", (d,)), (s + "norm2b", p + "post_ffw_norm.weight", "gain", (d,)),
                    (s + "mlp.gate", p + "ffn_gate.weight", "mat", (ff, d)), (s + "mlp.up", p + "ffn_up.weight", "mat", (ff, d)),
                    (s + "mlp.down", p + "ffn_down.weight", "mat", (d, ff))]
    return out


def weights_from_tensors(j: dict, tensors: Mapping[str, torch.Tensor]) -> ModelWeights:
    cfg = config_from_json(j)
    return named_weights(cfg, tensor_names(cfg), tensors)
