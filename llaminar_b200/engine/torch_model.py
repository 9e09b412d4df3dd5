"""Pure-PyTorch model runner with the same interface as :class:`CudaModel` (paged KV, ForwardBatch).

It is the CPU execution path (``-d cpu``) and lets the scheduler, prefix cache, speculative
decoding and the parallel layouts be tested without a GPU.  Math is fp32 on dequantised weights;
tensor-parallel ranks hold the same slices the GPU runner would (see parallel/tp_plan.py) and
sum the row-parallel partial results with ``torch.distributed`` (gloo on CPU).
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F

from ..models import gdn, mixers
from ..models.config import LatentAttention, LightningAttention, MatrixLSTM, ModelConfig
from ..models.reference import moe_route, rmsnorm, rope_split_half
from ..models.weights import ModelWeights
from ..parallel.tp_plan import TPPlan
from .cuda_model import ForwardBatch
from .kv_cache import PAGE_SIZE, PagedKVCache


class TorchPagedModel:
    def __init__(self, weights: ModelWeights, device="cpu", max_tokens: int = 4096, tp=None, layer_range=None,
                 with_head: bool = True, with_embed: bool = True, with_mtp: bool = True):
        self.cfg: ModelConfig = weights.config
        self.device = torch.device(device)
        self.tp = tp
        self.max_tokens = max_tokens
        c = self.cfg
        pl = self.plan = TPPlan.build(c, tp.size if tp else 1, tp.rank if tp else 0, getattr(tp, "moe_mode", "expert-parallel"))
        self.n_heads_local, self.n_kv_local = pl.n_heads_local, pl.n_kv_local
        self.layer_ids = list(range(*layer_range)) if layer_range else list(range(c.n_layers))
        D = c.head_dim
        self.kv_layer_shapes = None
        f = lambda name: weights[name].to_float().to(self.device)
        self.embed = f("token_embd.weight") if with_embed else None
        self.head = None
        if with_head:
            self.out_norm = f("output_norm.weight")
            head = weights.get("output.weight") or weights["token_embd.weight"]
            self.head = head.rows(pl.vocab_start, pl.vocab_stop).to_float().to(self.device)
            self.vocab_local = pl.vocab_stop - pl.vocab_start

        if c.has_mixers:
            if self.layer_ids != list(range(c.n_layers)):
                raise ValueError(f"a {c.arch} model cannot be cut into pipeline stages")
            self._init_attention_stack(f) if c.is_attention_stack else self._init_mixers(f)
            return
        kv_ids, gdn_ids = c.kv_layers(self.layer_ids), c.gdn_layers(self.layer_ids)

        def ffn(L, p):
            if c.is_moe:
                L["router"] = f(p + "ffn_gate_inp.weight")
                e0, e1 = pl.expert_start, pl.expert_stop
                L["e0"], L["e1"] = e0, e1
                L["wg"] = f(p + "ffn_gate_exps.weight")[e0:e1]
                L["wu"] = f(p + "ffn_up_exps.weight")[e0:e1]
                L["wd"] = f(p + "ffn_down_exps.weight")[e0:e1]
                if c.shared_expert_ff:                      # replicated on every rank, added after the experts' sum
                    L["sh"] = (f(p + "ffn_gate_shexp.weight"), f(p + "ffn_up_shexp.weight"), f(p + "ffn_down_shexp.weight"),
                               f(p + "ffn_gate_inp_shexp.weight").reshape(-1, 1))
                return
            L["wg"] = f(p + "ffn_gate.weight")[pl.ff_start:pl.ff_stop]
            L["wu"] = f(p + "ffn_up.weight")[pl.ff_start:pl.ff_stop]
            L["wd"] = f(p + "ffn_down.weight")[:, pl.ff_start:pl.ff_stop]

        def gdn_layer(i):
            """Linear-attention block: all key heads (q and k rows) plus this rank's value heads."""
            p = f"blk.{i}."
            L = {"attn_norm": f(p + "attn_norm.weight"), "ffn_norm": f(p + c.ffn_norm_name), "index": i,
                 "gdn_index": gdn_ids.index(i)}
            d, kd = c.ssm_state, c.gdn_key_dim
            v0, v1 = pl.gdn_v_start, pl.gdn_v_stop
            rows = torch.cat([torch.arange(2 * kd), 2 * kd + torch.arange(v0 * d, v1 * d)])
            L["wqkv"] = f(p + "attn_qkv.weight")[rows]
            L["conv_w"] = f(p + "ssm_conv1d.weight")[rows]
            L["wz"] = f(p + "attn_gate.weight")[v0 * d:v1 * d]
            L["walpha"], L["wbeta"] = f(p + "ssm_alpha.weight")[v0:v1], f(p + "ssm_beta.weight")[v0:v1]
            L["ssm_a"], L["dt_bias"] = f(p + "ssm_a")[v0:v1], f(p + "ssm_dt.bias")[v0:v1]
            L["ssm_norm"] = f(p + "ssm_norm.weight")
            L["wout"] = f(p + "ssm_out.weight")[:, v0 * d:v1 * d]
            ffn(L, p)
            return L

        def layer(i):
            if c.is_gdn_layer(i):
                return gdn_layer(i)
            p = f"blk.{i}."
            L = {"attn_norm": f(p + "attn_norm.weight"), "ffn_norm": f(p + c.ffn_norm_name), "index": i,
                 "kv_index": kv_ids.index(i) if i in kv_ids else None}
            qs, qe, ks, ke = pl.q_head_start * D, pl.q_head_stop * D, pl.kv_head_start * D, pl.kv_head_stop * D
            qw = 2 if c.attn_gate else 1                       # rows of a head: [query | gate]
            L["wq"], L["wk"], L["wv"] = f(p + "attn_q.weight")[qs * qw:qe * qw], f(p + "attn_k.weight")[ks:ke], f(p + "attn_v.weight")[ks:ke]
            L["wo"] = f(p + "attn_output.weight")[:, qs:qe]
            if c.qkv_bias:
                L["bq"], L["bk"], L["bv"] = f(p + "attn_q.bias")[qs:qe], f(p + "attn_k.bias")[ks:ke], f(p + "attn_v.bias")[ks:ke]
            if c.qk_norm:
                L["qn"], L["kn"] = f(p + "attn_q_norm.weight"), f(p + "attn_k_norm.weight")
            ffn(L, p)
            return L

        self.layers = [layer(i) for i in self.layer_ids]
        self.mtp_layers = []
        self.mtp_kv_base = len(kv_ids)                  # the NextN layers' K/V follow this stage's own layers in the cache
        self.n_kv_layers = len(kv_ids) + (c.nextn_layers if with_mtp else 0)
        # what the engine needs to size the linear-attention state pools of this stage (None: no such layers)
        self.hybrid_dims = None
        if gdn_ids:
            nv = pl.gdn_v_stop - pl.gdn_v_start
            self.hybrid_dims = dict(n_layers=len(gdn_ids), conv_dim=2 * c.gdn_key_dim + nv * c.ssm_state,
                                    conv_kernel=c.ssm_conv_kernel, n_v_heads=nv, d=c.ssm_state)
        for j in range(c.nextn_layers if with_mtp else 0):
            i = c.n_layers + j
            L = layer(i)
            p = f"blk.{i}.nextn."
            for k in ("eh_proj", "enorm", "hnorm", "shared_head_norm"):
                L[k] = f(p + k + ".weight")
            self.mtp_layers.append(L)

    def weight_bytes(self) -> int:
        return 0

    # -- layers of latent, grouped or lightning attention ----------------------------------------------------------
    def _init_attention_stack(self, f) -> None:
        c = self.cfg
        self.embed_norm = f("token_embd_norm.weight") if c.embed_norm else None
        self.loop_in = f("loop_in.weight") if c.loop else None
        self.loop_step = f("loop_step.weight") if c.loop_steps else None
        latent = {"qa": "attn_q_a", "qan": "attn_q_a_norm", "qb": "attn_q_b", "kva": "attn_kv_a", "kvan": "attn_kv_a_norm", "kb": "attn_k_b", "vb": "attn_v_b"}
        self.positions = f("position_embd.weight") if c.learned_positions else None
        dense = {"wu": "ffn_up", "wd": "ffn_down", **({} if c.ffn_act == "gelu_up" else {"wg": "ffn_gate"})}
        experts = {"router": "ffn_gate_inp", "wg": "ffn_gate_exps", "wu": "ffn_up_exps", "wd": "ffn_down_exps"}
        self.layers, n_states = [], 0
        for i in self.layer_ids:
            m, e = c.mixers[i], c.experts_of(i)
            want = {"attn_norm": "attn_norm", **({"post_attn": "post_attention_norm"} if c.post_norms else {})}
            if isinstance(m, LatentAttention):
                want.update(wo="attn_output", **latent, **({"sink": "attn_sinks"} if m.sinks else {}), **({"gate": "attn_gate"} if m.gated else {}))
            elif isinstance(m, LightningAttention):
                want.update(wq="lin_q", wk="lin_k", wv="lin_v", gate="lin_g", on="lin_norm", wo="lin_output")
            else:
                want.update(wq="attn_q", wk="attn_k", wv="attn_v", wo="attn_output")
                for on, names in ((m.gate, {"gate": "attn_gate"}), (m.qk_norm, {"qn": "attn_q_norm", "kn": "attn_k_norm"}), (m.temperature, {"temp": "attn_temperature"}),
                                  (m.conv, {"cq": "attn_q_conv", "ck": "attn_k_conv", "cv": "attn_v_conv"}), (m.value_mix, {"vmix": "attn_value_mix"})):
                    want.update(names if on else {})
            if c.ff_width(i) or e:
                want.update({"ffn_norm": "ffn_norm", **({"post_ffn": "post_ffw_norm"} if c.post_norms else {}), **(experts if e else dense)})
            if c.depth_average:
                want["depth"] = "depth_average"
            L = {k: f(f"blk.{i}.{n}.weight") for k, n in want.items()}
            if e:
                L["router_bias"] = f(f"blk.{i}.ffn_gate_inp.bias") if e.bias else 0.0
            L.update(index=i, mixer=m, experts=e, state=n_states)
            n_states += mixers.has_state(m)
            if not isinstance(m, LightningAttention):
                L["freqs"] = torch.tensor(m.rotary.frequencies(), dtype=torch.float64, device=self.device)
            self.layers.append(L)
        self.runs = c.layer_runs()
        self.kv_layer_shapes, self.state_shapes = mixers.mixer_kv_shapes(c), mixers.mixer_state_shapes(c)
        self.kv_index = mixers.run_kv_layers(c)
        self.n_kv_layers = self.mtp_kv_base = len(self.kv_layer_shapes)
        self.mtp_layers, self.hybrid_dims = [], None

    @staticmethod
    def _turn(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, interleaved: bool = False) -> torch.Tensor:
        """Rotate the leading 2 x cos.shape[-1] values of the last dimension, pair (i, i + half) or (2i, 2i + 1)."""
        half = cos.shape[-1]
        if interleaved:
            a, b = x[..., 0:2 * half:2], x[..., 1:2 * half:2]
            return torch.cat([torch.stack([a * cos - b * sin, b * cos + a * sin], dim=-1).flatten(-2), x[..., 2 * half:]], dim=-1)
        a, b = x[..., :half], x[..., half:2 * half]
        return torch.cat([a * cos - b * sin, b * cos + a * sin, x[..., 2 * half:]], dim=-1)

    @staticmethod
    def _first_key(p: int, m) -> int:
        """First position that a query at position p sees."""
        lo = max(0, p - m.window + 1) if m.window else 0
        return max(lo, p - p % m.chunk) if getattr(m, "chunk", 0) else lo

    def _unseen(self, p: torch.Tensor, keys: torch.Tensor, m) -> torch.Tensor:
        """[rows, keys] True where the row at position p does not see the key."""
        first = torch.tensor([self._first_key(x, m) for x in p.tolist()])
        return (keys[None, :] > p[:, None]) | (keys[None, :] < first[:, None])

    def _latent_attention(self, L, x: torch.Tensor, fb: ForwardBatch, kvl: torch.Tensor) -> torch.Tensor:
        """Queries in the latent space against the cached latents, sequence by sequence."""
        c, m = self.cfg, L["mixer"]
        T, rot_off = x.shape[0], -(-m.kv_rank // 8) * 8
        pos = fb.positions.long()
        ang = pos.double()[:, None] * L["freqs"]
        cos, sin = (ang.cos() * m.rotary.magnitude).float(), (ang.sin() * m.rotary.magnitude).float()
        q = (rmsnorm(x @ L["qa"].T, L["qan"], c.rms_eps) @ L["qb"].T).view(T, m.heads, m.dim + m.rot_dim)
        q_rot = self._turn(q[..., m.dim:], cos[:, None], sin[:, None], m.rotary.interleaved)
        q_lat = torch.einsum("thd,hdr->thr", q[..., :m.dim], L["kb"].view(m.heads, m.dim, m.kv_rank))
        down = x @ L["kva"].T
        sid = fb.seq_ids.long()
        page, off = fb.block_table.long()[sid, pos // PAGE_SIZE], pos % PAGE_SIZE
        row = torch.zeros(T, kvl.shape[-1])
        row[:, :m.kv_rank] = rmsnorm(down[:, :m.kv_rank], L["kvan"], c.rms_eps)
        row[:, rot_off:rot_off + m.rot_dim] = self._turn(down[:, m.kv_rank:], cos, sin, m.rotary.interleaved)
        kvl[page, off] = row.to(kvl.dtype)
        out = torch.empty(T, m.heads, m.kv_rank)
        for b in sid.unique().tolist():
            rows = (sid == b).nonzero(as_tuple=True)[0]
            p = pos[rows]
            keys = torch.arange(self._first_key(int(p.min()), m), int(p.max()) + 1)
            kv = kvl[fb.block_table.long()[b, keys // PAGE_SIZE], keys % PAGE_SIZE].float()
            s = torch.einsum("thr,sr->hts", q_lat[rows], kv[:, :m.kv_rank])
            s = (s + torch.einsum("the,se->hts", q_rot[rows], kv[:, rot_off:rot_off + m.rot_dim])) * m.scale
            s = s.masked_fill(self._unseen(p, keys, m)[None], float("-inf"))
            if m.sinks:                       # one more column that carries no value
                s = torch.cat([s, L["sink"][:, None, None].expand(-1, s.shape[1], 1)], dim=-1)
            w = torch.softmax(s, -1)[..., :len(keys)]
            out[rows] = torch.einsum("hts,sr->thr", w, kv[:, :m.kv_rank])
        v = torch.einsum("thr,hvr->thv", out, L["vb"].view(m.heads, m.vdim, m.kv_rank)).reshape(T, -1)
        if "gate" in L:
            v = v * torch.sigmoid(x @ L["gate"].T)
        return v @ L["wo"].T

    def _conv_rows(self, L, u: torch.Tensor, w: torch.Tensor, at: int, fb: ForwardBatch, kv: PagedKVCache) -> torch.Tensor:
        """The convolution of projected rows u [T, n], channels ``at`` and on of the layer's; w [n, taps].  The state keeps the last
        rows of a sequence, position p in place p mod taps."""
        taps, n, out = w.shape[1], u.shape[1], torch.empty_like(u)
        ring = kv.hybrid.layers[L["state"]][0][:, :, at:at + n]
        for r0, r1, slot, _ in gdn.batch_sequences(fb.seq_ids, fb.positions, fb.state_slots):
            p0 = int(fb.positions[r0])
            past = torch.tensor([p for p in range(p0 - taps + 1, p0)], dtype=torch.long)
            before = ring[slot, past % taps] * (past >= 0)[:, None]
            out[r0:r1] = mixers.short_conv(u[r0:r1], before, w.T)
            for r in range(max(r0, r1 - taps + 1), r1):
                ring[slot, (p0 + r - r0) % taps] = u[r]
        return out

    def _grouped_attention(self, L, x: torch.Tensor, fb: ForwardBatch, kvl: torch.Tensor, kv: PagedKVCache | None = None, shared: dict | None = None) -> torch.Tensor:
        """``shared``: what layers of one forward call hand on (the values that later ones mix in)."""
        c, m, T = self.cfg, L["mixer"], x.shape[0]
        pos, sid = fb.positions.long(), fb.seq_ids.long()
        ang = pos.double()[:, None] * L["freqs"]
        cos, sin = (ang.cos() * m.rotary.magnitude).float()[:, None], (ang.sin() * m.rotary.magnitude).float()[:, None]
        turn = lambda y: self._turn(y, cos, sin, m.rotary.interleaved)
        q, k, v = x @ L["wq"].T, x @ L["wk"].T, x @ L["wv"].T
        if m.conv:
            q, k, v = (self._conv_rows(L, u, L[w], at, fb, kv) for u, w, at in ((q, "cq", 0), (k, "ck", q.shape[1]), (v, "cv", q.shape[1] + k.shape[1])))
        q, k = q.view(T, m.heads, m.dim), k.view(T, m.kv_heads, m.dim)
        if m.qk_norm:
            q, k = rmsnorm(q, L["qn"], c.rms_eps), rmsnorm(k, L["kn"], c.rms_eps)
        q, k = turn(q), turn(k)
        if m.temperature:
            q = q * L["temp"][:, None]
        q = q.view(T, m.kv_heads, -1, m.dim)
        if m.value_mix:
            first = shared.setdefault("values", v)
            v = v if first is v else torch.lerp(v, first, L["vmix"])
        page, off = fb.block_table.long()[sid, pos // PAGE_SIZE], pos % PAGE_SIZE
        kvl[page, 0, :, off, :m.dim] = k.to(kvl.dtype)
        kvl[page, 1, :, off, :m.vdim] = v.view(T, m.kv_heads, m.vdim).to(kvl.dtype)
        out = torch.empty(T, m.heads, m.vdim)
        for b in sid.unique().tolist():
            rows = (sid == b).nonzero(as_tuple=True)[0]
            p = pos[rows]
            keys = torch.arange(self._first_key(int(p.min()), m), int(p.max()) + 1)
            pages, off = fb.block_table.long()[b, keys // PAGE_SIZE], keys % PAGE_SIZE
            K, V = kvl[pages, 0, :, off, :m.dim].float(), kvl[pages, 1, :, off, :m.vdim].float()                # [keys, kv heads, size]
            s = torch.einsum("tghd,sgd->ghts", q[rows], K) * m.scale
            if m.softcap:
                s = mixers.soft_cap(s, m.softcap)
            s = s.masked_fill(self._unseen(p, keys, m), float("-inf"))
            if m.null_key:                                                             # one more column that carries no value
                s = torch.cat([s, s.new_zeros(*s.shape[:3], 1)], dim=-1)
            w = torch.softmax(s, -1)[..., :len(keys)]
            out[rows] = torch.einsum("ghts,sgd->tghd", w, V).reshape(len(rows), m.heads, m.vdim)
        if m.gate:
            out = out * torch.sigmoid(x @ L["gate"].T).view(T, m.heads, -1)            # one per head or one per value
        return out.reshape(T, -1) @ L["wo"].T

    def _lightning(self, L, x: torch.Tensor, fb: ForwardBatch, kv: PagedKVCache) -> torch.Tensor:
        m, T = L["mixer"], x.shape[0]
        q, k, v = (F.silu(x @ L[n].T).view(T, m.heads, -1) for n in ("wq", "wk", "wv"))
        decay, (S,), o = torch.tensor(m.decay), kv.hybrid.layers[L["state"]], torch.empty_like(v)
        for r0, r1, slot, fresh in gdn.batch_sequences(fb.seq_ids, fb.positions, fb.state_slots):
            if fresh:
                S[slot].zero_()
            o[r0:r1] = mixers.retention_rows(q[r0:r1], k[r0:r1], v[r0:r1], decay, S[slot])
        return (rmsnorm(o.reshape(T, -1), L["on"], self.cfg.rms_eps) * torch.sigmoid(x @ L["gate"].T)) @ L["wo"].T

    def _routed_experts(self, L, x: torch.Tensor) -> torch.Tensor:
        e = L["experts"]
        z = x @ L["router"].T + L["router_bias"]
        if e.keep < e.groups:
            groups = z.view(-1, e.groups, e.n // e.groups).amax(-1).topk(e.keep, dim=-1).indices
            kept = torch.zeros(z.shape[0], e.groups, dtype=torch.bool).scatter_(1, groups, True)
            z = z.masked_fill(~kept.repeat_interleave(e.n // e.groups, dim=1), float("-inf"))
        best = z.topk(e.top, dim=-1)
        wt, out = torch.softmax(best.values, dim=-1), torch.zeros_like(x)
        if getattr(self, "expert_stats", None) is not None:
            self.expert_stats.record(L["index"], best.indices)
        for j in best.indices.unique().tolist():
            tok, slot = (best.indices == j).nonzero(as_tuple=True)
            g, u = x[tok] @ L["wg"][j].T, x[tok] @ L["wu"][j].T
            y = (mixers.limited_pair(g, u, e.limit) if e.limit else F.silu(g) * u) @ L["wd"][j].T
            out.index_add_(0, tok, y * wt[tok, slot].unsqueeze(-1))
        return out

    def _run_parallel_stack(self, fb: ForwardBatch, kv: PagedKVCache) -> torch.Tensor:
        """Mixer and feed-forward side by side on the same input, a weighted sum over depth behind every layer."""
        c, eps, shared = self.cfg, self.cfg.rms_eps, {}
        h = self.embed[fb.tokens.long()].float()
        if c.learned_positions:
            h = h + self.positions[fb.positions.long()]
        streams = [h]
        for r, L in enumerate(self.layers):
            x = rmsnorm(h, L["attn_norm"], eps)
            if isinstance(L["mixer"], LightningAttention):
                y = self._lightning(L, x, fb, kv)
            else:
                y = self._grouped_attention(L, x, fb, kv.layers[self.kv_index[r]], kv, shared)
            if "wu" in L:
                x = rmsnorm(h, L["ffn_norm"], eps)
                y = y + (self._routed_experts(L, x) if L["experts"] else F.gelu(x @ L["wu"].T, approximate="tanh") @ L["wd"].T)
            h = h + y
            if c.depth_average:
                streams.append(h)
                h = torch.einsum("j,jtd->td", L["depth"], torch.stack(streams))
            if getattr(self, "taps", None) is not None:
                self.taps[f"layer{r}"] = h.clone()
        return h

    def _run_attention_stack(self, fb: ForwardBatch, kv: PagedKVCache) -> torch.Tensor:
        if self.cfg.parallel_ff:
            return self._run_parallel_stack(fb, kv)
        c, eps, n_pass = self.cfg, self.cfg.rms_eps, 0
        act = F.silu if c.ffn_act == "silu" else lambda z: F.gelu(z, approximate="tanh")
        x0 = self.embed[fb.tokens.long()].float()
        if c.embed_norm:
            x0 = rmsnorm(x0, self.embed_norm, eps)
        h = x0
        for r, (i, starts_pass) in enumerate(self.runs):
            L = self.layers[i]
            if starts_pass:
                h = torch.cat([h, x0], dim=-1) @ self.loop_in.T
                if c.loop_steps:
                    h = h + self.loop_step[n_pass]
                n_pass += 1
            mix = self._latent_attention if isinstance(L["mixer"], LatentAttention) else self._grouped_attention
            h = h + rmsnorm(mix(L, rmsnorm(h, L["attn_norm"], eps), fb, kv.layers[self.kv_index[r]]), L["post_attn"], eps)
            if "wg" in L:
                x = rmsnorm(h, L["ffn_norm"], eps)
                y = self._routed_experts(L, x) if L["experts"] else (act(x @ L["wg"].T) * (x @ L["wu"].T)) @ L["wd"].T
                h = h + rmsnorm(y, L["post_ffn"], eps)
            if getattr(self, "taps", None) is not None:
                self.taps[f"layer{r}"] = h.clone()
        return h

    # -- layers of windowed attention, retention and matrix LSTMs --------------------------------------------
    def _init_mixers(self, f) -> None:
        c = self.cfg
        self.side_embed = f("side_embd.weight") if c.side_dim else None
        self.layers, kv_i, st_i = [], 0, 0
        for i in self.layer_ids:
            p, m = f"blk.{i}.", c.mixers[i]
            L = {"mixer": m, "state": st_i, "kv": kv_i, "post_mix": f(p + "post_attention_norm.weight") * f(p + "post_attention_scale.weight")}
            names = ["lstm_q", "lstm_k", "lstm_v", "lstm_g", "lstm_i", "lstm_f", "lstm_output", "lstm_norm"] if isinstance(m, MatrixLSTM) else \
                ["attn_q", "attn_k", "attn_gate", "attn_q_norm", "attn_k_norm", "attn_sinks", "attn_output", "attn_out_norm",
                 "ret_q", "ret_k", "ret_v", "ret_g", "ret_output", "ret_out_norm"]
            L.update({n: f(f"{p}{n}.weight") for n in names})
            if isinstance(m, MatrixLSTM):
                L["bi"], L["bf"] = f(p + "lstm_i.bias"), f(p + "lstm_f.bias")
            else:
                L["freqs"] = torch.tensor(m.right.rotary.frequencies(), dtype=torch.float64, device=self.device)
                kv_i += 1
            st_i += 1
            if c.ff_width(i):
                L["post_ffn"] = f(p + "post_ffw_norm.weight") * f(p + "post_ffw_scale.weight")
                L["wu"], L["wd"] = f(p + "ffn_up.weight"), f(p + "ffn_down.weight")
            if c.side_dim:
                L.update({n: f(f"{p}{n}.weight") for n in ("side_gate", "side_proj", "side_norm")})
            self.layers.append(L)
        self.kv_layer_shapes = mixers.mixer_kv_shapes(c)
        self.state_shapes = mixers.mixer_state_shapes(c)
        self.n_kv_layers = self.mtp_kv_base = len(self.kv_layer_shapes)
        self.mtp_layers, self.hybrid_dims = [], None

    def _recurrent(self, L, m, q, k, v, fb: ForwardBatch, kv: PagedKVCache, rows_fn) -> torch.Tensor:
        """Runs `rows_fn(q, k, v, first row, end row, *state)` per sequence on its slot's state; returns the heads' outputs, each
        divided by its root mean square."""
        state, out = kv.hybrid.layers[L["state"]], torch.empty_like(v)
        for r0, r1, slot, fresh in gdn.batch_sequences(fb.seq_ids, fb.positions, fb.state_slots):
            if fresh:
                for t in state:
                    t[slot].zero_()
            out[r0:r1] = rows_fn(q[r0:r1], k[r0:r1], v[r0:r1], r0, r1, *(t[slot] for t in state))
        return (out * torch.rsqrt(out.pow(2).mean(-1, keepdim=True) + self.cfg.rms_eps)).reshape(q.shape[0], -1)

    def _mlstm(self, L, x: torch.Tensor, fb: ForwardBatch, kv: PagedKVCache) -> torch.Tensor:
        m, T = L["mixer"], x.shape[0]
        q, k, v = ((x @ L[f"lstm_{n}"].T).view(T, m.heads, -1) for n in "qkv")
        i, f = mixers.mlstm_gates(x @ L["lstm_i"].T + L["bi"], x @ L["lstm_f"].T + L["bf"], m.gate_cap)
        o = self._recurrent(L, m, q * m.dim ** -0.5, k, v, fb, kv, lambda q, k, v, r0, r1, *st: mixers.mlstm_rows(q, k, v, i[r0:r1], f[r0:r1], *st))
        return (o * L["lstm_norm"] * torch.sigmoid(x @ L["lstm_g"].T)) @ L["lstm_output"].T

    def _retention(self, L, x: torch.Tensor, fb: ForwardBatch, kv: PagedKVCache) -> torch.Tensor:
        m, T = L["mixer"].right, x.shape[0]
        q, k, v = ((x @ L[f"ret_{n}"].T).view(T, m.heads, -1) for n in "qkv")
        ang = fb.positions.double()[:, None] * L["freqs"]
        cos, sin = ang.cos().float()[:, None], ang.sin().float()[:, None]
        q, k = self._turn(q, cos, sin), self._turn(k, cos, sin) * m.dim ** -0.5
        decay = torch.tensor(m.decay)
        o = self._recurrent(L, m, q, k, v, fb, kv, lambda q, k, v, r0, r1, S: mixers.retention_rows(q, k, v, decay, S))
        return (o * F.silu(x @ L["ret_g"].T)) @ L["ret_output"].T

    def _window_attention(self, L, x: torch.Tensor, fb: ForwardBatch, kvl: torch.Tensor) -> torch.Tensor:
        c, m, T = self.cfg, L["mixer"].left, x.shape[0]
        k = x @ L["attn_k"].T
        v = k.view(T, m.kv_heads, m.dim)
        q = rmsnorm(x @ L["attn_q"].T, L["attn_q_norm"], c.rms_eps).view(T, m.kv_heads, -1, m.dim)
        k = rmsnorm(k, L["attn_k_norm"], c.rms_eps).view(T, m.kv_heads, m.dim)
        pos, sid = fb.positions.long(), fb.seq_ids.long()
        page, off = fb.block_table.long()[sid, pos // PAGE_SIZE], pos % PAGE_SIZE
        kvl[page, 0, :, off], kvl[page, 1, :, off] = k.to(kvl.dtype), v.to(kvl.dtype)
        out = torch.empty(T, m.heads * m.dim)
        for b in sid.unique().tolist():
            rows = (sid == b).nonzero(as_tuple=True)[0]
            p = pos[rows]
            keys = torch.arange(max(0, int(p.min()) - m.window + 1) if m.window else 0, int(p.max()) + 1)
            pages, off = fb.block_table.long()[b, keys // PAGE_SIZE], keys % PAGE_SIZE
            K, V = kvl[pages, 0, :, off].float(), kvl[pages, 1, :, off].float()                # [keys, kv heads, dim]
            s = torch.einsum("tghd,sgd->ghts", q[rows], K) * m.scale
            hidden = keys[None, :] > p[:, None]
            if m.window:
                hidden |= keys[None, :] <= p[:, None] - m.window
            s = s.masked_fill(hidden, float("-inf"))
            sink = L["attn_sinks"].view(m.kv_heads, -1, 1, 1).expand(*s.shape[:3], 1)          # one more column that carries no value
            w = torch.softmax(torch.cat([s, sink], dim=-1), -1)[..., :-1]
            out[rows] = torch.einsum("ghts,sgd->tghd", w, V).reshape(len(rows), -1)
        return (out * torch.sigmoid(x @ L["attn_gate"].T)) @ L["attn_output"].T

    def _run_mixers(self, fb: ForwardBatch, kv: PagedKVCache) -> torch.Tensor:
        c, eps = self.cfg, self.cfg.rms_eps
        tok = fb.tokens.long()
        h = self.embed[tok].float() * c.embed_scale
        norm = lambda x, w: F.layer_norm(x, x.shape[-1:], w, None, eps)
        for i, L in enumerate(self.layers):
            if isinstance(L["mixer"], MatrixLSTM):
                y = self._mlstm(L, h, fb, kv)
            else:
                y = 0.5 * (rmsnorm(self._window_attention(L, h, fb, kv.layers[L["kv"]]), L["attn_out_norm"], eps)
                           + rmsnorm(self._retention(L, h, fb, kv), L["ret_out_norm"], eps))
            h = h + c.residual_mult * norm(y, L["post_mix"])
            if "wu" in L:
                h = h + c.residual_mult * norm(F.relu(h @ L["wu"].T).square() @ L["wd"].T, L["post_ffn"])
            if c.side_dim:
                e = self.side_embed[tok, i * c.side_dim:(i + 1) * c.side_dim]
                y = (F.gelu(h @ L["side_gate"].T, approximate="tanh") * e) @ L["side_proj"].T
                h = h + c.residual_mult * rmsnorm(y, L["side_norm"], eps)
            if getattr(self, "taps", None) is not None:
                self.taps[f"layer{i}"] = h.clone()
        return h

    # ---------------------------------------------------------------------------------------
    def _sum_ranks(self, x: torch.Tensor) -> torch.Tensor:
        if self.tp is not None and self.tp.size > 1:
            self.tp.all_reduce(x)
        return x

    def _attention(self, L, x, fb: ForwardBatch, kvl: torch.Tensor) -> torch.Tensor:
        c = self.cfg
        T, D = x.shape[0], c.head_dim
        q, k, v = x @ L["wq"].T, x @ L["wk"].T, x @ L["wv"].T
        if c.qkv_bias:
            q, k, v = q + L["bq"], k + L["bk"], v + L["bv"]
        gate = None
        if c.attn_gate:
            q, gate = q.view(T, self.n_heads_local, 2, D).unbind(dim=2)
            gate = gate.reshape(T, -1)
        q = q.reshape(T, self.n_heads_local, D)
        k = k.view(T, self.n_kv_local, D)
        v = v.view(T, self.n_kv_local, D)
        if c.qk_norm:
            q, k = rmsnorm(q, L["qn"], c.rms_eps), rmsnorm(k, L["kn"], c.rms_eps)
        pos = fb.positions.long()
        q, k = rope_split_half(q, pos, c.rope_theta, c.rotary_dim), rope_split_half(k, pos, c.rope_theta, c.rotary_dim)
        sid = fb.seq_ids.long()
        page = fb.block_table.long()[sid, pos // PAGE_SIZE]
        off = pos % PAGE_SIZE
        kvl[page, 0, :, off] = k.to(kvl.dtype)
        kvl[page, 1, :, off] = v.to(kvl.dtype)
        g = self.n_heads_local // self.n_kv_local
        out = torch.empty(T, self.n_heads_local, D, dtype=torch.float32, device=x.device)
        scale = 1.0 / math.sqrt(D)
        for b in sid.unique().tolist():
            rows = (sid == b).nonzero(as_tuple=True)[0]
            last = int(pos[rows].max())
            n_pages = last // PAGE_SIZE + 1
            pages = fb.block_table.long()[b, :n_pages]
            K = kvl[pages, 0].permute(1, 0, 2, 3).reshape(self.n_kv_local, n_pages * PAGE_SIZE, D)[:, :last + 1].float()
            V = kvl[pages, 1].permute(1, 0, 2, 3).reshape(self.n_kv_local, n_pages * PAGE_SIZE, D)[:, :last + 1].float()
            K, V = K.repeat_interleave(g, 0), V.repeat_interleave(g, 0)
            s = torch.einsum("thd,hsd->hts", q[rows], K) * scale
            mask = torch.arange(last + 1, device=x.device)[None, :] > pos[rows][:, None]
            s = s.masked_fill(mask[None], float("-inf"))
            out[rows] = torch.einsum("hts,hsd->thd", torch.softmax(s, -1), V)
        out = out.reshape(T, -1)
        if gate is not None:
            out = out * torch.sigmoid(gate)
        return out @ L["wo"].T

    def _linear_attention(self, L, x, fb: ForwardBatch, kv: PagedKVCache) -> torch.Tensor:
        c, hs, gi = self.cfg, kv.hybrid, L["gdn_index"]
        nv = self.plan.gdn_v_stop - self.plan.gdn_v_start
        if fb.defer_state:                       # speculative verification: R rows per sequence, state committed afterwards
            B = fb.state_slots.shape[0]
            sh = lambda t: t.view(B, x.shape[0] // B, -1)
            rows, hs.stash[gi] = gdn.gdn_rows_deferred(sh(x @ L["wqkv"].T), sh(x @ L["wz"].T), sh(x @ L["walpha"].T), sh(x @ L["wbeta"].T),
                                                       L["conv_w"], L["ssm_a"], L["dt_bias"], L["ssm_norm"], hs.conv[gi], hs.rec[gi],
                                                       fb.state_slots.long(), c.ssm_k_heads, nv, c.ssm_state, c.rms_eps,
                                                       self.plan.gdn_v_start)
            hs.stash_slots = fb.state_slots.long()
            return rows @ L["wout"].T
        seqs = gdn.batch_sequences(fb.seq_ids, fb.positions, fb.state_slots)
        rows = gdn.gdn_block_rows(x @ L["wqkv"].T, x @ L["wz"].T, x @ L["walpha"].T, x @ L["wbeta"].T, seqs,
                                  hs.conv[gi], hs.rec[gi], L["conv_w"], L["ssm_a"], L["dt_bias"], L["ssm_norm"],
                                  c.ssm_k_heads, self.plan.gdn_v_stop - self.plan.gdn_v_start, c.ssm_state, c.rms_eps,
                                  self.plan.gdn_v_start)
        return rows @ L["wout"].T

    def _ffn(self, L, x: torch.Tensor) -> torch.Tensor:
        c = self.cfg
        if not c.is_moe:
            return (F.silu(x @ L["wg"].T) * (x @ L["wu"].T)) @ L["wd"].T
        idx, wt = moe_route(x @ L["router"].T, c.n_experts_used, c.norm_topk_prob)
        if getattr(self, "expert_stats", None) is not None:
            self.expert_stats.record(L["index"], idx)
        out = torch.zeros_like(x)
        for e in range(L["e0"], L["e1"]):
            tok, slot = (idx == e).nonzero(as_tuple=True)
            if tok.numel() == 0:
                continue
            le = e - L["e0"]
            xe = x[tok]
            ye = (F.silu(xe @ L["wg"][le].T) * (xe @ L["wu"][le].T)) @ L["wd"][le].T
            out.index_add_(0, tok, ye * wt[tok, slot].unsqueeze(-1))
        return out

    def _layer(self, L, h, fb, kvl, kv=None):
        c = self.cfg
        x = rmsnorm(h, L["attn_norm"], c.rms_eps)
        h = h + self._sum_ranks(self._linear_attention(L, x, fb, kv) if "gdn_index" in L else self._attention(L, x, fb, kvl))
        xn = rmsnorm(h, L["ffn_norm"], c.rms_eps)
        y = self._ffn(L, xn)
        if not (c.is_moe and getattr(self.tp, "moe_mode", "expert-parallel") == "replicated"):
            y = self._sum_ranks(y)               # replicated experts: every rank already has the full sum
        if "sh" in L:
            wg, wu, wd, gate = L["sh"]
            y = y + torch.sigmoid(xn @ gate) * ((F.silu(xn @ wg.T) * (xn @ wu.T)) @ wd.T)
        return h + y

    def _logits(self, h_rows, norm_w, out):
        x = F.layer_norm(h_rows, h_rows.shape[-1:], norm_w, None, self.cfg.rms_eps) if self.cfg.norm_kind == "layer" else rmsnorm(h_rows, norm_w, self.cfg.rms_eps)
        lg = x @ self.head.T * self.cfg.logit_scale
        if out is not None:
            out[:lg.shape[0]].copy_(lg)
            return out[:lg.shape[0]]
        return lg

    @torch.no_grad()
    def forward(self, fb: ForwardBatch, kv: PagedKVCache, logits_out=None, want_logits=True, kv_layer_offset: int = 0):
        own = self.cfg.has_mixers
        if own:
            h = self._run_attention_stack(fb, kv) if self.cfg.is_attention_stack else self._run_mixers(fb, kv)
        else:
            h = fb.embeds.float() if fb.embeds is not None else self.embed[fb.tokens.long()].float()
        for li, L in enumerate(() if own else self.layers):
            kvl = kv.layers[kv_layer_offset + L["kv_index"]] if L.get("kv_index") is not None else None
            h = self._layer(L, h, fb, kvl, kv)
            if getattr(self, "taps", None) is not None:       # per-layer hidden states for the parity report
                self.taps[f"layer{li}"] = h.float().clone()
        logits = None
        if want_logits and self.head is not None:
            rows = h if fb.logit_rows is None else h.index_select(0, fb.logit_rows.long())
            logits = self._logits(rows, self.out_norm, logits_out)
        return logits, h

    @torch.no_grad()
    def mtp_forward(self, fb: ForwardBatch, hidden: torch.Tensor, kv: PagedKVCache, depth: int = 0, logits_out=None):
        c = self.cfg
        L = self.mtp_layers[depth]
        e = rmsnorm(self.embed[fb.tokens.long()].float(), L["enorm"], c.rms_eps)
        hn = rmsnorm(hidden.float(), L["hnorm"], c.rms_eps)
        x = torch.cat([e, hn], dim=-1) @ L["eh_proj"].T
        h = self._layer(L, x, fb, kv.layers[self.mtp_kv_base + depth])
        rows = h if fb.logit_rows is None else h.index_select(0, fb.logit_rows.long())
        return self._logits(rows, L["shared_head_norm"], logits_out), h
