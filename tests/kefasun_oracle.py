"""Plain, slow implementation of the Kefasun decoder, one function per mechanism, for comparison with the engine.

Works on one sequence of token ids at a time, whole prompts only: no cache, no batching, no rearrangement of weights (keys and
values of the latent layers are written out per head, every expert runs on its own tokens).  `model` is a dictionary
{"config": config.json as a dict, "tensors": name -> tensor}; everything runs in the dtype of ``dt`` (float64 by default, so that
the oracle adds no rounding of its own).
"""
from __future__ import annotations

import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def angles(positions, rot, dt):
    """Cosine and sine [n, dims / 2] of position x frequency."""
    freqs = torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)], dtype=torch.float64)
    a = torch.tensor([float(p) for p in positions], dtype=torch.float64)[:, None] * freqs
    return a.cos().to(dt), a.sin().to(dt)


def rotate_neighbours(x, positions, rot):
    """x [..., n, size]: values 2i and 2i + 1 of the first `dims` turn together."""
    cos, sin = angles(positions, rot, x.dtype)
    out = x.clone()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2], out[..., 1:rot["dims"]:2] = u * cos - v * sin, v * cos + u * sin
    return out


def rotate_halves(x, positions, rot):
    """x [..., n, size]: values i and i + dims / 2 turn together."""
    cos, sin = angles(positions, rot, x.dtype)
    half = rot["dims"] // 2
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, rest], dim=-1)


def causal_mask(n):
    """[n, n] True where query i sees key j."""
    return torch.arange(n)[None, :] <= torch.arange(n)[:, None]


def window_mask(n, size):
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return causal_mask(n) & (i - j < size)


def chunk_mask(n, size):
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return causal_mask(n) & (i // size == j // size)


def mask_size(m):
    return (m.get("mask") or {}).get("size")


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def softmax_with_sink(scores, sink):
    """scores [H, n, n] (-inf where unseen), sink [H]: exp(sink) joins the denominator."""
    top = torch.maximum(scores.max(dim=-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(scores - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def softmax_plus_one(scores):
    return softmax_with_sink(scores, torch.zeros(scores.shape[0], dtype=scores.dtype))


def plain_softmax(scores):
    return torch.softmax(scores, dim=-1)


def head_gate(o, z):
    """o [n, H, vdim], z [n, H]: one factor per head."""
    return o * torch.sigmoid(z)[..., None]


def value_gate(o, z):
    """o [n, H, vdim], z [n, H * vdim]: one factor per value."""
    return o * torch.sigmoid(z).reshape(o.shape)


def grouped_heads(h, m, T, eps, rotate):
    """Queries [H, n, dim], keys [H, n, dim] and values [H, n, vdim], every key head repeated for its query heads."""
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms_norm((h @ T("q").T).reshape(n, H, m["dim"]), T("q.norm"), eps).transpose(0, 1)
    k = rms_norm((h @ T("k").T).reshape(n, G, m["dim"]), T("k.norm"), eps).transpose(0, 1)
    v = (h @ T("v").T).reshape(n, G, m["vdim"]).transpose(0, 1)
    q, k = rotate(q, range(n), m["rot"]), rotate(k, range(n), m["rot"])
    owner = [i // (H // G) for i in range(H)]
    return q, k[owner], v[owner]


def chunked_attention(h, m, T, eps):
    """Type 'attention': neighbours rotate, a query sees its own chunk, one joins the denominator, one gate per head."""
    n = h.shape[0]
    q, k, v = grouped_heads(h, m, T, eps, rotate_neighbours)
    size = mask_size(m)
    seen = chunk_mask(n, size) if size else causal_mask(n)
    s = (q @ k.transpose(1, 2) * m["scale"]).masked_fill(~seen[None], float("-inf"))
    o = (softmax_plus_one(s) @ v).transpose(0, 1)
    return head_gate(o, h @ T("g").T).reshape(n, -1) @ T("o").T


def capped_attention(h, m, T, eps):
    """Type 'attention_2': halves rotate, scores are soft-capped, every earlier key is seen, one gate per value."""
    n = h.shape[0]
    q, k, v = grouped_heads(h, m, T, eps, rotate_halves)
    s = q @ k.transpose(1, 2) * m["scale"]
    if m.get("softcap"):
        s = soft_cap(s, m["softcap"])
    o = (plain_softmax(s.masked_fill(~causal_mask(n)[None], float("-inf"))) @ v).transpose(0, 1)
    return value_gate(o, h @ T("g").T).reshape(n, -1) @ T("o").T


def latent_attention(h, m, T, eps):
    n, H = h.shape[0], m["heads"]
    dim, rd, vd, rank = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = rms_norm(h @ T("dq").T, T("dq.norm"), eps) @ T("uq").T
    q = q.reshape(n, H, dim + rd).transpose(0, 1)
    down = h @ T("dkv").T
    c, kr = rms_norm(down[:, :rank], T("dkv.norm"), eps), down[:, rank:]
    k = (c @ T("uk").T).reshape(n, H, dim).transpose(0, 1)
    v = (c @ T("uv").T).reshape(n, H, vd).transpose(0, 1)
    qr, kr = rotate_neighbours(q[..., dim:], range(n), m["rot"]), rotate_neighbours(kr, range(n), m["rot"])
    s = (q[..., :dim] @ k.transpose(1, 2) + qr @ kr.T) * m["scale"]
    seen = window_mask(n, mask_size(m)) if mask_size(m) else causal_mask(n)
    o = (softmax_with_sink(s.masked_fill(~seen[None], float("-inf")), T("sink")) @ v).transpose(0, 1)
    return value_gate(o, h @ T("g").T).reshape(n, -1) @ T("o").T


MIXERS = {"attention": chunked_attention, "latent_attention": latent_attention, "attention_2": capped_attention}


def gated_ffn(h, T):
    return (silu(h @ T("gate").T) * (h @ T("up").T)) @ T("down").T


def route(h, T, top):
    """Experts [n, top] with the largest logits and the softmax over just those."""
    z = h @ T("router").T + T("router.b")
    best = z.topk(top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def router_gap(h, T, top):
    """[n] distance between the last logit that is chosen and the first that is not (infinite when all are)."""
    z = torch.cat([h @ T("router").T + T("router.b"), h.new_full((h.shape[0], 1), float("-inf"))], dim=-1).sort(dim=-1, descending=True).values
    return z[:, top - 1] - z[:, top]


def experts_ffn(h, m, T):
    ids, weights = route(h, T, m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        y = gated_ffn(h, lambda name: T(f"e{e}.{name}"))
        out = out + y * (weights * (ids == e)).sum(-1, keepdim=True)
    return out


def decoder_layer(x, i, model, W, gaps=None):
    entry, eps, p = model["config"]["layers"][i], model["config"]["norm"]["eps"], f"l{i}."
    mix, mlp = (lambda name: W(p + "mix." + name)), (lambda name: W(p + "mlp." + name))
    y = MIXERS[entry["type"]](rms_norm(x, W(p + "norm1"), eps), entry["mixer"], mix, eps)
    x = x + rms_norm(y, W(p + "norm1b"), eps)
    f = entry.get("mlp")
    if f:
        h = rms_norm(x, W(p + "norm2"), eps)
        if gaps is not None and f["kind"] == "moe":
            gaps.append(router_gap(h, mlp, f["router"]["top"]))
        y = gated_ffn(h, mlp) if f["kind"] == "dense" else experts_ffn(h, f, mlp)
        x = x + rms_norm(y, W(p + "norm2b"), eps)
    return x


def enter_pass(x, x0, t, W):
    return torch.cat([x, x0], dim=-1) @ W("loop.in").T + W("loop.step")[t]


def run_order(cfg):
    """(layer, number of the pass that starts with it or None) of every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    start, stop, times = (loop["start"], loop["stop"], loop["times"]) if loop else (n, n, 0)
    out = [(i, None) for i in range(start)]
    for t in range(times):
        out += [(i, t if i == start else None) for i in range(start, stop)]
    return out + [(i, None) for i in range(stop, n)]


def forward(tokens, model, dt=torch.float64, taps=None, gaps=None):
    """Logits [n, vocab] of one sequence; `taps` (a list) receives the residual stream after every layer run, `gaps` how close every
    choice of experts was."""
    cfg = model["config"]
    W = lambda name: model["tensors"][name].to(dt)
    x = x0 = W("embed")[torch.as_tensor(tokens).long()]
    for i, t in run_order(cfg):
        if t is not None:
            x = enter_pass(x, x0, t, W)
        x = decoder_layer(x, i, model, W, gaps)
        if taps is not None:
            taps.append(x)
    return rms_norm(x, W("final.norm"), cfg["norm"]["eps"]) @ W("embed").T * cfg["logit_scale"]


# -- models --------------------------------------------------------------------------------------------------------------------
def random_model(layers, seed=0, vocab=97, width=48, loop=None, eps=1e-5, sink_shift=0.0, gain=1.0, logit_scale=0.7):
    """A small model with random weights of the given layer list (see the `*_entry` functions)."""
    g = torch.Generator().manual_seed(seed)
    t = {}

    def mat(name, n, k, s=1.0):
        t[name] = (torch.randn(n, k, generator=g) * s * gain / math.sqrt(k)).to(torch.bfloat16)

    def vec(name, n, mean=0.0, s=0.2):
        t[name] = (torch.randn(n, generator=g) * s + mean).to(torch.bfloat16)

    def ffn(p, ff):
        mat(p + "gate", ff, width, 1.5), mat(p + "up", ff, width), mat(p + "down", width, ff)

    t["embed"] = torch.randn(vocab, width, generator=g).to(torch.bfloat16)
    if loop:
        mat("loop.in", width, 2 * width, 1.4)
        t["loop.step"] = (torch.randn(loop["times"], width, generator=g) * 0.7).to(torch.bfloat16)
    for i, e in enumerate(layers):
        m, p = e["mixer"], f"l{i}."
        H, dim, vd = m["heads"], m["dim"], m["vdim"]
        vec(p + "norm1", width, 1.0), vec(p + "norm1b", width, 1.0)
        if e["type"] == "latent_attention":
            rd, r = m["rot_dim"], m["kv_rank"]
            mat(p + "mix.dq", m["q_rank"], width), vec(p + "mix.dq.norm", m["q_rank"], 1.0)
            mat(p + "mix.uq", H * (dim + rd), m["q_rank"], 1.5)
            mat(p + "mix.dkv", r + rd, width), vec(p + "mix.dkv.norm", r, 1.0)
            mat(p + "mix.uk", H * dim, r, 1.5), mat(p + "mix.uv", H * vd, r)
            vec(p + "mix.sink", H, sink_shift, 1.0)
        else:
            G = m["kv_heads"]
            mat(p + "mix.q", H * dim, width), mat(p + "mix.k", G * dim, width), mat(p + "mix.v", G * vd, width)
            vec(p + "mix.q.norm", dim, 1.2, 0.4), vec(p + "mix.k.norm", dim, 1.2, 0.4)
        mat(p + "mix.g", H if e["type"] == "attention" else H * vd, width, 1.5)
        mat(p + "mix.o", width, H * vd)
        f = e.get("mlp")
        if f:
            vec(p + "norm2", width, 1.0), vec(p + "norm2b", width, 1.0)
            if f["kind"] == "dense":
                ffn(p + "mlp.", f["ff"])
            else:
                n = f["router"]["experts"]
                mat(p + "mlp.router", n, width, 3.0), vec(p + "mlp.router.b", n, 0.0, 0.5)
                for x in range(n):
                    ffn(f"{p}mlp.e{x}.", f["expert"]["ff"])
    vec("final.norm", width, 1.0)
    cfg = {"architecture": "Kefasun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_scale": logit_scale}
    if loop:
        cfg["loop"] = loop
    return {"config": cfg, "tensors": t}


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=40):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def chunked_entry(heads=4, kv_heads=2, dim=24, vdim=16, rot_dims=8, chunk=20, scale=None, base=1000.0, mlp=dense()):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk} if chunk else None,
                      "rot": {"base": base, "dims": rot_dims}, "scale": scale if scale is not None else dim ** -0.5}}


def capped_entry(heads=4, kv_heads=2, dim=16, vdim=24, rot_dims=16, softcap=8.0, scale=None, base=5000.0, mlp=dense()):
    return {"type": "attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "softcap": softcap,
                      "rot": {"base": base, "dims": rot_dims}, "scale": scale if scale is not None else dim ** -0.5}}


def latent_entry(heads=3, dim=24, rot_dim=8, vdim=16, kv_rank=40, q_rank=32, window=20, scale=None, base=1000.0, mlp=dense()):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "mask": {"size": window} if window else None, "rot": {"base": base, "dims": rot_dim},
                      "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}}
