"""Plain, slow implementation of the Pozivik decoder, one function per mechanism, for comparison with the engine.

Works on one sequence of token ids at a time, whole prompts only: no cache, no batching, no low-rank rearrangement (keys and
values are always written out per head).  `model` is a dictionary {"config": config.json as a dict, "tensors": name -> tensor};
everything runs in the dtype of ``dt`` (float64 by default, so that the oracle adds no rounding of its own).
"""
from __future__ import annotations

import math

import torch


def rms_divide(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def plain_norm(x, w, eps):
    return rms_divide(x, eps) * w


def centred_norm(x, w, eps):
    """The stored weight is the distance of the gain from one."""
    return rms_divide(x, eps) * (1 + w)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotation_frequencies(rot):
    """Angle per position of every pair, and the factor on sine and cosine."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    freqs, magnitude = [], 1.0
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            where = lambda turns: dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
            lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / sc["factor"] * ramp + f * (1 - ramp)
        freqs.append(f)
    if sc:
        magnitude = 0.1 * math.log(sc["factor"]) + 1
    return freqs, magnitude


def rotate(x, positions, rot):
    """x [..., T, n]: the pairs (i, i + dims/2) of the first `dims` values turn by position x frequency."""
    freqs, magnitude = rotation_frequencies(rot)
    half = len(freqs)
    ang = torch.tensor([[float(p) * f for f in freqs] for p in positions], dtype=torch.float64)
    cos, sin = (ang.cos() * magnitude).to(x.dtype), (ang.sin() * magnitude).to(x.dtype)
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, rest], dim=-1)


def window_mask(n, size):
    """[n, n] True where query i sees key j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    if size:
        seen = seen & (i - j < size)
    return seen


def softmax_with_sink(scores, sink):
    """scores [H, n, n] (-inf where unseen), sink [H]: exp(sink) joins the denominator."""
    top = torch.maximum(scores.max(dim=-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(scores - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def latent_attention(h, m, T, eps, positions=None):
    """h [n, width]; m: the mixer's entry of the configuration; T(name): its tensors."""
    n, H = h.shape[0], m["heads"]
    dim, rd, vd, rank = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = list(range(n)) if positions is None else positions
    q = plain_norm(h @ T("dq").T, T("dq.norm"), eps) @ T("uq").T
    q = q.reshape(n, H, dim + rd).transpose(0, 1)                       # [H, n, dim + rd]
    down = h @ T("dkv").T
    c, kr = plain_norm(down[:, :rank], T("dkv.norm"), eps), down[:, rank:]
    k = (c @ T("uk").T).reshape(n, H, dim).transpose(0, 1)
    v = (c @ T("uv").T).reshape(n, H, vd).transpose(0, 1)
    qr, kr = rotate(q[..., dim:], positions, m["rot"]), rotate(kr, positions, m["rot"])
    s = (q[..., :dim] @ k.transpose(1, 2) + qr @ kr.T) * m["scale"]
    size = (m.get("mask") or {}).get("size")
    s = s.masked_fill(~window_mask(n, size)[None], float("-inf"))
    o = softmax_with_sink(s, T("sink")) @ v
    return o.transpose(0, 1).reshape(n, H * vd) @ T("o").T


def feed_forward(h, T):
    return (gelu_tanh(h @ T("gate").T) * (h @ T("up").T)) @ T("down").T


def decoder_layer(x, i, model, W):
    entry, eps = model["config"]["layers"][i], model["config"]["norm"]["eps"]
    p = f"l{i}."
    y = latent_attention(centred_norm(x, W(p + "norm1"), eps), entry["mixer"], lambda n: W(p + "mix." + n), eps)
    x = x + centred_norm(y, W(p + "norm1b"), eps)
    if entry.get("mlp"):
        y = feed_forward(centred_norm(x, W(p + "norm2"), eps), lambda n: W(p + "mlp." + n))
        x = x + centred_norm(y, W(p + "norm2b"), eps)
    return x


def forward(tokens, model, dt=torch.float64, taps=None):
    """Logits [n, vocab] of one sequence; `taps` (a list) receives the residual stream after every layer run."""
    cfg = model["config"]
    W = lambda name: model["tensors"][name].to(dt)
    eps = cfg["norm"]["eps"]
    x0 = centred_norm(W("embed")[torch.as_tensor(tokens).long()], W("embed.norm"), eps)
    x, n = x0, len(cfg["layers"])
    loop = cfg.get("loop")

    def run(i, x):
        x = decoder_layer(x, i, model, W)
        if taps is not None:
            taps.append(x)
        return x

    start, stop, times = (loop["start"], loop["stop"], loop["times"]) if loop else (n, n, 0)
    for i in range(start):
        x = run(i, x)
    for _ in range(times):
        x = torch.cat([x, x0], dim=-1) @ W("loop.in").T
        for i in range(start, stop):
            x = run(i, x)
    for i in range(stop, n):
        x = run(i, x)
    return centred_norm(x, W("final.norm"), eps) @ W("head").T


def random_model(seed=0, vocab=97, width=48, layers=None, loop=None, eps=1e-5, sink_shift=0.0, gain=1.0):
    """A small model with random weights of the given layer list (see `layer_entry`)."""
    g = torch.Generator().manual_seed(seed)
    t = {}

    def mat(name, n, k, s=1.0):
        t[name] = (torch.randn(n, k, generator=g) * s * gain / math.sqrt(k)).to(torch.bfloat16)

    def vec(name, n, mean=0.0, s=0.2):
        t[name] = (torch.randn(n, generator=g) * s + mean).to(torch.bfloat16)

    t["embed"] = torch.randn(vocab, width, generator=g).to(torch.bfloat16)
    vec("embed.norm", width)
    if loop:
        mat("loop.in", width, 2 * width)
    for i, e in enumerate(layers):
        m, p = e["mixer"], f"l{i}."
        H, dim, rd, vd, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        vec(p + "norm1", width), vec(p + "norm1b", width)
        mat(p + "mix.dq", m["q_rank"], width), vec(p + "mix.dq.norm", m["q_rank"], 1.0)
        mat(p + "mix.uq", H * (dim + rd), m["q_rank"], 1.5)
        mat(p + "mix.dkv", r + rd, width), vec(p + "mix.dkv.norm", r, 1.0)
        mat(p + "mix.uk", H * dim, r, 1.5), mat(p + "mix.uv", H * vd, r)
        vec(p + "mix.sink", H, sink_shift, 1.0)
        mat(p + "mix.o", width, H * vd)
        if e.get("mlp"):
            ff = e["mlp"]["ff"]
            vec(p + "norm2", width), vec(p + "norm2b", width)
            mat(p + "mlp.gate", ff, width), mat(p + "mlp.up", ff, width), mat(p + "mlp.down", width, ff)
    vec("final.norm", width)
    mat("head", vocab, width)
    cfg = {"architecture": "Pozivik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        cfg["loop"] = loop
    return {"config": cfg, "tensors": t}


def layer_entry(heads=3, dim=24, rot_dim=8, vdim=16, kv_rank=40, q_rank=32, window=20, scale=None, base=1000.0, scaling=None, ff=56):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "mask": {"size": window}, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5,
                      "rot": {"base": base, "dims": rot_dim, **({"scaling": scaling} if scaling else {})}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def save(model, folder):
    """Writes config.json and model.safetensors (the container format: u64 header length, JSON header, data)."""
    import json
    import os
    import struct
    names = {torch.bfloat16: "BF16", torch.float32: "F32", torch.int32: "I32"}
    header, blobs, at = {}, [], 0
    for name, x in model["tensors"].items():
        b = x.contiguous().flatten().view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[x.dtype], "shape": list(x.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(model["config"], f)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
