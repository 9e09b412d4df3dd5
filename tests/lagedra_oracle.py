"""Plain, slow implementation of the Lagedra decoder, one function per mechanism, for comparison with the engine.

Works on one sequence of token ids at a time, whole prompts only: no cache, no batching, no rearrangement of weights (the recurrence
runs token by token, every expert on every token).  `model` is a dictionary {"config": config.json as a dict, "tensors": name ->
tensor}; everything runs in the dtype of ``dt`` (float64 by default, so that the oracle adds no rounding of its own).
"""
from __future__ import annotations

import math

import torch


def scalar_norm(x, gain, eps):
    """One gain for all values."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * gain


def gain_norm(x, w, eps):
    """A gain per value."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def add_positions(x, table):
    return x + table[:x.shape[0]]


# -- linear attention ------------------------------------------------------------------------------------------------------------
def decayed_state(q, k, v, decay):
    """q, k [n, H, d], v [n, H, e], decay [H] -> [n, H, e], one token after the other."""
    n, H, d = q.shape
    S, out = torch.zeros(H, d, v.shape[2], dtype=q.dtype), torch.empty_like(v)
    for t in range(n):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hde,hd->he", S, q[t])
    return out


def output_gate(o, z):
    return o * torch.sigmoid(z)


def lightning(h, m, T, eps, values):
    n, H = h.shape[0], m["heads"]
    q, k = (silu(h @ T(x).T).reshape(n, H, m["dim"]) for x in "qk")
    v = silu(h @ T("v").T).reshape(n, H, m["vdim"])
    o = decayed_state(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)).reshape(n, -1)
    return output_gate(gain_norm(o, T("norm"), eps), h @ T("g").T) @ T("o").T


# -- attention -------------------------------------------------------------------------------------------------------------------
def short_conv(u, w):
    """u [n, channels], w [channels, taps]: every channel over its own last `taps` values, zeros in front."""
    n, taps = u.shape[0], w.shape[1]
    padded = torch.cat([u.new_zeros(taps - 1, u.shape[1]), u])
    return sum(w[:, j] * padded[j:j + n] for j in range(taps))


def yarn(rot):
    """Frequencies of the pairs and the factor on cosine and sine."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not s:
        return freqs, 1.0
    where = lambda turns: dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), dims - 1)
    ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]
    return [f / s["factor"] * r + f * (1 - r) for f, r in zip(freqs, ramp)], 0.1 * math.log(s["factor"]) + 1


def rotate_halves(x, positions, rot):
    """x [..., n, size]: values i and i + dims / 2 of the first dims turn together."""
    freqs, grow = yarn(rot)
    a = torch.tensor([float(p) for p in positions], dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)
    cos, sin = (a.cos() * grow).to(x.dtype), (a.sin() * grow).to(x.dtype)
    half = rot["dims"] // 2
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, rest], dim=-1)


def window_mask(n, size):
    """[n, n] True where query i sees key j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (i - j >= 0) & ((i - j < size) if size else True)


def head_temperature(s, temp):
    return s * temp[:, None, None]


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def mix_values(v, first, share):
    """A token's values in the earlier layer take their share of this layer's."""
    return v if first is None else (1 - share) * v + share * first


def mask_size(m):
    return (m.get("mask") or {}).get("size")


def owner(heads, kv_heads):
    return [i // (heads // kv_heads) for i in range(heads)]


def attention(h, m, T, eps, values):
    """``values``: {"first": values of the first layer that mixes}, filled here."""
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (short_conv(h @ T(x).T, T(x + ".conv")) for x in "qkv")
    q, k = (rotate_halves(x.reshape(n, -1, m["dim"]).transpose(0, 1), range(n), m["rot"]) for x in (q, k))
    if m.get("v_mix"):
        first = values.get("first")
        values.setdefault("first", v)
        v = mix_values(v, first, T("vmix"))
    of = owner(H, G)
    k, v = k[of], v.reshape(n, G, m["vdim"]).transpose(0, 1)[of]
    s = head_temperature(q @ k.transpose(1, 2) * m["scale"], T("temp"))
    if m.get("softcap"):
        s = soft_cap(s, m["softcap"])
    w = torch.softmax(s.masked_fill(~window_mask(n, mask_size(m)), float("-inf")), dim=-1)
    return (w @ v).transpose(0, 1).reshape(n, -1) @ T("o").T


MIXERS = {"attention": attention, "lightning": lightning}


# -- feed-forward ----------------------------------------------------------------------------------------------------------------
def plain_ffn(h, T):
    return gelu_tanh(h @ T("up").T) @ T("down").T


def limited_ffn(h, T, limit):
    g = (h @ T("gate").T).clamp(max=limit)
    u = (h @ T("up").T).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ T("down").T


def allowed_experts(s, groups):
    """s [n, experts] -> True where an expert's group is among the best ones (by its best score)."""
    if not groups:
        return torch.ones_like(s, dtype=torch.bool)
    best = s.reshape(s.shape[0], groups["count"], -1).amax(-1)
    keep = torch.zeros_like(best, dtype=torch.bool).scatter(1, best.topk(groups["keep"], dim=-1).indices, True)
    return keep.repeat_interleave(s.shape[1] // groups["count"], dim=1)


def expert_weights(s, ids):
    chosen = s.gather(1, ids)
    return chosen / (chosen.sum(-1, keepdim=True) + 1e-20)


def route(h, T, router):
    """Chosen experts [n, top] and their weights."""
    s = torch.softmax(h @ T("router").T, dim=-1)
    ids = s.masked_fill(~allowed_experts(s, router.get("groups")), -1.0).topk(router["top"], dim=-1).indices
    return ids, expert_weights(s, ids)


def router_gap(h, T, router):
    """[n] how far (in logits) the choices of experts and of groups are from turning out otherwise."""
    z = h @ T("router").T
    low = z.new_full((z.shape[0], 1), float("-inf"))

    def gap(x, n):
        x = torch.cat([x, low], dim=-1).sort(dim=-1, descending=True).values
        return x[:, n - 1] - x[:, n]

    g = router.get("groups")
    out = gap(z.masked_fill(~allowed_experts(torch.softmax(z, -1), g), float("-inf")), router["top"])
    return torch.minimum(out, gap(z.reshape(z.shape[0], g["count"], -1).amax(-1), g["keep"])) if g else out


def experts_ffn(h, m, T):
    ids, weights = route(h, T, m["router"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        y = limited_ffn(h, lambda name: T(f"e{e}.{name}"), m["expert"]["limit"])
        out = out + y * (weights * (ids == e)).sum(-1, keepdim=True)
    return out


# -- the decoder -----------------------------------------------------------------------------------------------------------------
def depth_average(xs, w):
    return sum(w[j] * x for j, x in enumerate(xs))


def layer_result(x, i, model, W, values, gaps=None):
    entry, eps, p = model["config"]["layers"][i], model["config"]["norm"]["eps"], f"l{i}."
    mix, mlp = (lambda name: W(p + "mix." + name)), (lambda name: W(p + "mlp." + name))
    y = MIXERS[entry["type"]](scalar_norm(x, W(p + "norm1"), eps), entry["mixer"], mix, eps, values)
    f = entry.get("mlp")
    if f:
        h = scalar_norm(x, W(p + "norm2"), eps)
        if gaps is not None and f["kind"] == "moe":
            gaps.append(router_gap(h, mlp, f["router"]))
        y = y + (plain_ffn(h, mlp) if f["kind"] == "dense" else experts_ffn(h, f, mlp))
    return x + y


def forward(tokens, model, dt=torch.float64, taps=None, gaps=None):
    """Logits [n, vocab] of one sequence; `taps` (a list) receives the residual stream after every layer, `gaps` how close every
    choice of experts was."""
    cfg = model["config"]
    W = lambda name: model["tensors"][name].to(dt)
    x = add_positions(W("embed")[torch.as_tensor(tokens).long()], W("pos"))
    xs, values = [x], {}
    for i in range(len(cfg["layers"])):
        xs.append(layer_result(x, i, model, W, values, gaps))
        x = depth_average(xs, W(f"l{i}.dwa"))
        if taps is not None:
            taps.append(x)
    return scalar_norm(x, W("final.norm"), cfg["norm"]["eps"]) @ W("head").T


# -- models --------------------------------------------------------------------------------------------------------------------
def random_model(layers, seed=0, vocab=97, width=48, eps=1e-5, gain=1.0, max_positions=700):
    """A small model with random weights of the given layer list (see the `*_entry` functions)."""
    g = torch.Generator().manual_seed(seed)
    bf, t = torch.bfloat16, {}
    rnd = lambda *s: torch.randn(*s, generator=g)

    def mat(name, n, k, s=1.0):
        t[name] = (rnd(n, k) * s * gain / math.sqrt(k)).to(bf)

    def num(name, mean=1.0, s=0.3):
        t[name] = (rnd(1)[0] * s + mean).to(bf)

    t["embed"], t["pos"] = rnd(vocab, width).to(bf), (0.5 * rnd(max_positions, width)).to(bf)
    for i, e in enumerate(layers):
        m, p = e["mixer"], f"l{i}."
        H, dim, vd = m["heads"], m["dim"], m["vdim"]
        num(p + "norm1")
        if e["type"] == "lightning":
            mat(p + "mix.q", H * dim, width, 1.5), mat(p + "mix.k", H * dim, width, 1.5), mat(p + "mix.v", H * vd, width, 1.5)
            mat(p + "mix.g", H * vd, width, 1.5)
            t[p + "mix.norm"] = (rnd(H * vd) * 0.3 + 1.0).to(bf)
        else:
            G = m["kv_heads"]
            for x, n in (("q", H * dim), ("k", G * dim), ("v", G * vd)):
                mat(f"{p}mix.{x}", n, width, 1.5 if x != "v" else 1.0)
                t[f"{p}mix.{x}.conv"] = (rnd(n, m["conv"]) * 0.5 + (torch.arange(m["conv"]) == m["conv"] - 1)).to(bf)
            t[p + "mix.temp"] = (rnd(H) * 0.4 + 1.2).to(bf)
            if m.get("v_mix"):
                num(p + "mix.vmix", 0.75, 0.1)
        mat(p + "mix.o", width, H * vd)
        f = e.get("mlp")
        if f:
            num(p + "norm2")
            if f["kind"] == "dense":
                mat(p + "mlp.up", f["ff"], width, 1.5), mat(p + "mlp.down", width, f["ff"])
            else:
                n, ff = f["router"]["experts"], f["expert"]["ff"]
                mat(p + "mlp.router", n, width, 3.0)
                for x in range(n):
                    mat(f"{p}mlp.e{x}.gate", ff, width, 1.5), mat(f"{p}mlp.e{x}.up", ff, width, 1.5), mat(f"{p}mlp.e{x}.down", width, ff)
        w = rnd(i + 2) * 0.2
        w[i + 1] += 1.0
        t[p + "dwa"] = w.to(bf)
    num("final.norm")
    mat("head", vocab, width)
    return {"config": {"architecture": "Lagedra", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "max_positions": max_positions}, "tensors": t}


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=40, count=2, keep=1, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def lightning_entry(heads=3, dim=24, vdim=16, decay=(0.7, 0.95, 0.998), mlp=dense()):
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)[:heads]}}


def attention_entry(heads=4, kv_heads=2, dim=24, vdim=16, rot_dims=16, window=20, conv=4, softcap=6.0, scale=None, base=1000.0, scaling="yarn", v_mix=True, mlp=dense()):
    scaling = {"factor": 5.0, "original": 200, "fast": 16.0, "slow": 1.0} if scaling == "yarn" else scaling
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": window} if window else None,
                      "rot": {"base": base, "dims": rot_dims, "scaling": scaling}, "scale": scale if scale is not None else dim ** -0.5, "softcap": softcap, "v_mix": v_mix}}
