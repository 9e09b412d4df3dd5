"""Plain, slow implementation of the Zogepel decoder, one function per mechanism, for comparison with the engine.

Works on one sequence of token ids at a time, whole prompts only: no cache, no batching; recurrences run token by token.
`model` is a dictionary {"config": config.json as a dict, "tensors": name -> tensor}; everything runs in the dtype of ``dt``
(float64 by default, so that the oracle adds no rounding of its own).
"""
from __future__ import annotations

import math

import torch


# -- norms and activations -----------------------------------------------------------------------------------------------------
def rms_divide(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_divide(x, eps) * w


def layer_norm(x, w, eps):
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def squared_relu(z):
    return torch.clamp(z, min=0) ** 2


def silu(z):
    return z * torch.sigmoid(z)


# -- positions and masks -------------------------------------------------------------------------------------------------------
def rotate(x, positions, dims, base):
    """x [T, H, n]: the pairs (i, i + dims/2) of the first `dims` values turn by position x base^(-2i/dims)."""
    half = dims // 2
    freqs = [base ** (-2.0 * i / dims) for i in range(half)]
    ang = torch.tensor([[float(p) * f for f in freqs] for p in positions], dtype=torch.float64)
    cos, sin = ang.cos().to(x.dtype)[:, None], ang.sin().to(x.dtype)[:, None]
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, rest], dim=-1)


def window_mask(n, size):
    """[n, n] True where query i sees key j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & (i - j < size)


def softmax_with_sink(scores, sink):
    """scores [H, n, n] (-inf where unseen), sink [H]: exp(sink) joins the denominator."""
    top = torch.maximum(scores.max(dim=-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(scores - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


# -- recurrences ---------------------------------------------------------------------------------------------------------------
def mlstm_gates(h, wi, bi, wf, bf, cap):
    """Log input gate and log forget gate [T, H]."""
    soft = lambda z: cap * torch.tanh(z / cap)
    return soft(h @ wi.T + bi), -torch.log1p(torch.exp(-soft(h @ wf.T + bf)))


def mlstm_scan(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, e], log gates i, f [T, H] -> o [T, H, e]."""
    T, H, d = q.shape
    S, n, m = q.new_zeros(H, d, v.shape[-1]), q.new_zeros(H, d), q.new_zeros(H)
    out = []
    for t in range(T):
        top = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - top), torch.exp(i[t] - top)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = top
        size = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[t]) / size[:, None])
    return torch.stack(out)


def retention_scan(q, k, v, decay):
    T, H, d = q.shape
    S, out = q.new_zeros(H, d, v.shape[-1]), []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out)


# -- mixers --------------------------------------------------------------------------------------------------------------------
def heads_of(x, n):
    return x.reshape(x.shape[0], n, -1)


def mlstm(h, m, T, eps):
    H = m["heads"]
    q, k, v = (heads_of(h @ T(x).T, H) for x in "qkv")
    i, f = mlstm_gates(h, T("i"), T("i.b"), T("f"), T("f.b"), m["gate_cap"])
    o = rms_divide(mlstm_scan(q * m["dim"] ** -0.5, k, v, i, f), eps).reshape(h.shape[0], -1)
    return (o * T("norm") * torch.sigmoid(h @ T("g").T)) @ T("o").T


def key_value_attention(h, m, T, eps):
    """Sliding-window attention whose values are the projected keys before their norm."""
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    k = h @ T("k").T
    v = heads_of(k, G)
    q, k = heads_of(rms_norm(h @ T("q").T, T("q.norm"), eps), H), heads_of(rms_norm(k, T("k.norm"), eps), G)
    of = [x // (H // G) for x in range(H)]
    s = torch.einsum("thd,shd->hts", q, k[:, of]) * m["scale"]
    s = s.masked_fill(~window_mask(n, m["mask"]["size"])[None], float("-inf"))
    o = torch.einsum("hts,shd->thd", softmax_with_sink(s, T("sink")), v[:, of]).reshape(n, -1)
    return (o * torch.sigmoid(h @ T("g").T)) @ T("o").T


def retention(h, m, T, eps):
    H, pos = m["heads"], range(h.shape[0])
    q, k, v = (heads_of(h @ T(x).T, H) for x in "qkv")
    q, k = (rotate(x, pos, m["rot"]["dims"], m["rot"]["base"]) for x in (q, k))
    o = retention_scan(q, k * m["dim"] ** -0.5, v, torch.tensor(m["decay"], dtype=h.dtype))
    return (rms_divide(o, eps).reshape(h.shape[0], -1) * silu(h @ T("g").T)) @ T("o").T


def parallel(h, m, T, eps):
    left = key_value_attention(h, m["left"], lambda n: T("left." + n), eps)
    right = retention(h, m["right"], lambda n: T("right." + n), eps)
    return 0.5 * (rms_norm(left, T("left.out"), eps) + rms_norm(right, T("right.out"), eps))


# -- the decoder ---------------------------------------------------------------------------------------------------------------
def feed_forward(x, T):
    return squared_relu(x @ T("up").T) @ T("down").T


def side_input(x, e, T, eps):
    return rms_norm((gelu_tanh(x @ T("gate").T) * e) @ T("proj").T, T("norm"), eps)


def decoder_layer(x, i, e, model, W):
    cfg = model["config"]
    entry, eps, mult, p = cfg["layers"][i], cfg["norm"]["eps"], cfg["residual_mult"], f"l{i}."
    mixer = {"mlstm": mlstm, "parallel": parallel}[entry["type"]]
    y = mixer(x, entry["mixer"], lambda n: W(p + "mix." + n), eps)
    x = x + mult * layer_norm(y, W(p + "norm1"), eps) * W(p + "ls1")
    if entry.get("mlp"):
        y = feed_forward(x, lambda n: W(p + "mlp." + n))
        x = x + mult * layer_norm(y, W(p + "norm2"), eps) * W(p + "ls2")
    return x + mult * side_input(x, e, lambda n: W(p + "side." + n), eps)


def forward(tokens, model, dt=torch.float64, taps=None):
    """Logits [n, vocab] of one sequence; `taps` (a list) receives the residual stream after every layer."""
    cfg = model["config"]
    W = lambda name: model["tensors"][name].to(dt)
    ids, dim = torch.as_tensor(tokens).long(), cfg["token_side"]["dim"]
    x, side = W("embed")[ids] * cfg["embedding"]["scale"], W("side.embed")[ids]
    for i in range(len(cfg["layers"])):
        x = decoder_layer(x, i, side[:, i * dim:(i + 1) * dim], model, W)
        if taps is not None:
            taps.append(x)
    return layer_norm(x, W("final.norm"), cfg["norm"]["eps"]) @ W("head").T


# -- small random models -------------------------------------------------------------------------------------------------------
def random_model(seed=0, vocab=97, width=48, layers=None, eps=1e-5, mult=0.4, embed_scale=3.0, side_dim=10, sink_shift=0.0, gain=1.0):
    g = torch.Generator().manual_seed(seed)
    t = {}

    def mat(name, n, k, s=1.0):
        t[name] = (torch.randn(n, k, generator=g) * s * gain / math.sqrt(k)).to(torch.bfloat16)

    def vec(name, n, mean=1.0, s=0.2):
        t[name] = (torch.randn(n, generator=g) * s + mean).to(torch.bfloat16)

    t["embed"] = (torch.randn(vocab, width, generator=g) / embed_scale).to(torch.bfloat16)
    t["side.embed"] = torch.randn(vocab, side_dim * len(layers), generator=g).to(torch.bfloat16)
    for i, e in enumerate(layers):
        m, p = e["mixer"], f"l{i}."
        vec(p + "norm1", width), vec(p + "ls1", width)
        if e["type"] == "mlstm":
            H, d, ve = m["heads"], m["dim"], m["vdim"]
            mat(p + "mix.q", H * d, width, 1.5), mat(p + "mix.k", H * d, width, 1.5), mat(p + "mix.v", H * ve, width)
            # a query lies along its own key: with n.q near zero the normaliser turns the sign of a rounding error into the output's
            t[p + "mix.q"] = (0.6 * t[p + "mix.q"].float() + 0.8 * t[p + "mix.k"].float()).to(torch.bfloat16)
            mat(p + "mix.g", H * ve, width), mat(p + "mix.o", width, H * ve), vec(p + "mix.norm", H * ve)
            mat(p + "mix.i", H, width), vec(p + "mix.i.b", H, -1.0, 1.0)
            mat(p + "mix.f", H, width), vec(p + "mix.f.b", H, 3.0, 1.5)
        else:
            a, r = m["left"], m["right"]
            H, G, d = a["heads"], a["kv_heads"], a["dim"]
            q = p + "mix.left."
            mat(q + "q", H * d, width), mat(q + "k", G * d, width), mat(q + "g", H * d, width), mat(q + "o", width, H * d)
            vec(q + "q.norm", H * d, 1.5), vec(q + "k.norm", G * d, 1.5), vec(q + "sink", H, sink_shift, 1.0), vec(q + "out", width)
            H, d, ve = r["heads"], r["dim"], r["vdim"]
            q = p + "mix.right."
            mat(q + "q", H * d, width), mat(q + "k", H * d, width), mat(q + "v", H * ve, width)
            mat(q + "g", H * ve, width), mat(q + "o", width, H * ve), vec(q + "out", width)
        if e.get("mlp"):
            ff = e["mlp"]["ff"]
            vec(p + "norm2", width), vec(p + "ls2", width)
            mat(p + "mlp.up", ff, width), mat(p + "mlp.down", width, ff)
        mat(p + "side.gate", side_dim, width), mat(p + "side.proj", width, side_dim), vec(p + "side.norm", width)
    vec("final.norm", width)
    mat("head", vocab, width)
    cfg = {"architecture": "Zogepel", "embedding": {"scale": embed_scale}, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult,
           "token_side": {"dim": side_dim}, "vocab": vocab, "width": width}
    return {"config": cfg, "tensors": t}


def mlstm_layer(heads=3, dim=24, vdim=16, cap=10.0, ff=56):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def parallel_layer(heads=4, kv_heads=2, dim=24, window=20, scale=None, r_heads=3, r_dim=20, r_vdim=28, r_rot=12, base=1000.0, decay=None, ff=56):
    decay = decay or [1 - 2.0 ** (-5 - i) for i in range(r_heads)]
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": window}, "scale": scale if scale is not None else dim ** -0.5},
                      "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": decay, "rot": {"base": base, "dims": r_rot}}},
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
