"""Model hyper-parameters read from GGUF metadata, plus the named benchmark shapes.

Keys follow the ``<arch>.*`` convention the reference extracts (reference:
src/v2/loaders/ModelLoader.cpp:2548-2652) and the MoE / NextN keys it uses
(src/v2/models/qwen35moe/Qwen35MoEGraphConfigBuilder.cpp:37-45,
src/v2/execution/mtp/MTPWeightManifest.cpp:141-156).
"""
from __future__ import annotations

import json
import math
from dataclasses import asdict, dataclass, field, replace

from ..gguf.constants import GGMLType

SUPPORTED_ARCHS = ("qwen2", "qwen3", "qwen3moe", "qwen35", "qwen35moe", "pozivik", "zogepel", "kefasun", "lagedra")


@dataclass(frozen=True)
class RopeScaling:
    """YaRN: pairs that turn less than `slow` times over the original context are slowed down by `factor`, pairs that turn
    more than `fast` times keep their frequency, the ones between are blended; sine and cosine grow by a common factor."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotary:
    """Rotation of the first `dims` values of a vector by position x frequency i: pair (i, i + dims/2), or (2i, 2i + 1) when
    `interleaved`."""
    dims: int
    base: float
    scaling: RopeScaling | None = None
    interleaved: bool = False

    def frequencies(self) -> list[float]:
        """Angle per position of each of the dims/2 pairs (double precision)."""
        plain = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        s = self.scaling
        if s is None:
            return plain

        def pair_with(turns: float) -> float:
            """The (fractional) pair index that completes `turns` turns over the original context."""
            return self.dims * math.log(s.original / (turns * 2.0 * math.pi)) / (2.0 * math.log(self.base))

        first = max(math.floor(pair_with(s.fast)), 0)
        last = min(math.ceil(pair_with(s.slow)), self.dims - 1)
        out = []
        for i, f in enumerate(plain):
            slowed = min(1.0, max(0.0, (i - first) / max(last - first, 0.001)))
            out.append(f * (1.0 - slowed) + f * slowed / s.factor)
        return out

    def halves_order(self, size: int) -> list[int]:
        """Order of a vector's `size` values in which pair i is (i, i + dims/2).  Queries and keys in the same order have the same
        products, so projections can be stored in it and only one layout reaches the kernels."""
        if not self.interleaved:
            return list(range(size))
        return list(range(0, self.dims, 2)) + list(range(1, self.dims, 2)) + list(range(self.dims, size))

    @property
    def magnitude(self) -> float:
        return 1.0 if self.scaling is None else 1.0 + 0.1 * math.log(self.scaling.factor)


@dataclass(frozen=True)
class LatentAttention:
    """Attention over a low-rank latent: the cache holds one normed latent of `kv_rank` values and one rotated key part of
    `rot_dim` values per token, shared by all heads; per-head keys (`dim` unrotated values) and values (`vdim`) are linear
    functions of the latent.  Queries pass through a latent of `q_rank` values."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rotary: Rotary
    window: int = 0                 # keys a query sees, itself included (0: all before it)
    sinks: bool = True              # one learned logit per head in the softmax denominator
    gated: bool = False             # heads times sigmoid of a projection of the input, value by value, before the output projection

    @property
    def cache_width(self) -> int:
        """Values of a token's cache row: the latent and the rotated part, each starting on a 16-byte boundary in 16-bit
        form, padded to whole 16-value MMA steps."""
        return (-(-self.kv_rank // 8) * 8 + -(-self.rot_dim // 8) * 8 + 15) // 16 * 16


@dataclass(frozen=True)
class GroupedAttention:
    """Grouped-query softmax attention with per-head keys and values in the paged cache.  Queries and keys are rotated, in front of
    that RMS-normed per head (one gain per value, shared by the heads) or passed through a short causal convolution per channel."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rotary: Rotary
    window: int = 0                 # keys a query sees, itself included (0: all before it)
    chunk: int = 0                  # a query sees keys of its own chunk of positions only (0: no chunks)
    softcap: float = 0.0            # scores s become softcap * tanh(s / softcap) (0: as they are)
    null_key: bool = False          # one joins the softmax denominator (a key with score 0 and no value)
    gate: str = ""                  # "head" | "value": sigmoid of a projection of the input, per head or per value, before the output projection
    qk_norm: bool = True
    conv: int = 0                   # taps of the convolution over time on the projected queries, keys and values (0: none)
    temperature: bool = False       # one learned factor per query head on the scores, before the soft cap
    value_mix: bool = False         # a token's values in the first layer that has this join those of the later ones, with a learned share

    @property
    def head_size(self) -> int:
        """Values of a head in the cache, where keys and values have rows of one length."""
        return max(self.dim, self.vdim)

    @property
    def gate_width(self) -> int:
        return {"": 0, "head": self.heads, "value": self.heads * self.vdim}[self.gate]


@dataclass(frozen=True)
class Experts:
    """Mixture-of-experts feed-forward: the `top` experts with the largest router logits, weighted by the softmax over just those (or
    over all experts and divided by the chosen ones' sum: the same weights).  With several `groups` of neighbours only experts of
    the `keep` groups whose best experts are largest can be chosen.

    An expert is silu(gate) * up, or with a `limit` g sigmoid(1.702 g) (u + 1) of g = min(gate, limit) and u = up clamped to
    [-limit, limit]."""
    n: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1
    limit: float = 0.0
    bias: bool = True               # on the router logits


@dataclass(frozen=True)
class WindowAttention:
    """Grouped-query softmax attention with per-head keys and values in the paged cache, no rotation.  Queries and keys are
    RMS-normed over the whole projection (all heads together, one gain per value)."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int = 0                 # keys a query sees, itself included (0: all before it)
    sinks: bool = True              # one learned logit per head in the softmax denominator
    tied_values: bool = True        # the values are the projected keys before their norm
    gated: bool = True              # heads times sigmoid of a projection of the input, before the output projection


@dataclass(frozen=True)
class Retention:
    """Linear attention S_t = decay_h S_(t-1) + k_t v_t^T with rotated queries and keys, no denominator; the output of a head is
    divided by its root mean square and gated by silu."""
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]        # per head
    rotary: Rotary


@dataclass(frozen=True)
class LightningAttention:
    """Linear attention S_t = decay_h S_(t-1) + k_t v_t^T with silu on queries, keys and values, no rotation, scale or denominator;
    one RMS norm (a gain per value) spans the outputs of all heads, a sigmoid gates them."""
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]        # per head


@dataclass(frozen=True)
class MatrixLSTM:
    """Linear attention with exponential input gate and logistic forget gate per head and token (mLSTM): state S [dim, vdim], the
    normaliser n [dim] and the running maximum of the log gates.  Both gates are soft-capped; the output of a head is divided by
    its root mean square, scaled by a gain per value and gated by a sigmoid."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ParallelMixers:
    """Two mixers on the same input; half the sum of their outputs, each RMS-normed over the model width."""
    left: WindowAttention
    right: Retention


def mixer_parts(m) -> tuple:
    """The elementary mixers of a layer."""
    return (m.left, m.right) if isinstance(m, ParallelMixers) else (m,)


@dataclass
class ModelConfig:
    arch: str = "qwen3"
    n_layers: int = 2
    d_model: int = 256
    n_heads: int = 4
    n_kv_heads: int = 2
    head_dim: int = 64
    d_ff: int = 768
    vocab_size: int = 1024
    rope_theta: float = 1e6
    rms_eps: float = 1e-6
    context_length: int = 4096
    qk_norm: bool = True            # qwen3 / qwen3moe: per-head RMSNorm on Q and K
    qkv_bias: bool = False          # qwen2: biases on the Q/K/V projections
    tie_embeddings: bool = True
    # MoE
    n_experts: int = 0
    n_experts_used: int = 0
    expert_ff: int = 0
    norm_topk_prob: bool = True
    shared_expert_ff: int = 0       # qwen35moe: one always-on expert of this width, scaled by sigmoid(x . ffn_gate_inp_shexp)
    # multi-token prediction (NextN) head: number of extra decoder layers stored after the trunk
    nextn_layers: int = 0
    # hybrid layout (qwen35): every `full_attention_interval`-th layer is softmax attention over the KV cache, the others are
    # Gated-DeltaNet linear attention (short causal convolution + one recurrent d_k x d_v state per value head)
    # (reference: src/v2/models/qwen35/Qwen35GraphConfigBuilder.cpp:56-137)
    full_attention_interval: int = 0     # 0: every layer is full attention
    ssm_conv_kernel: int = 4
    ssm_state: int = 0                   # d_k = d_v of the linear-attention heads
    ssm_k_heads: int = 0
    ssm_v_heads: int = 0
    rope_dim: int = 0                    # leading dims of each head that are rotated (0: all of head_dim)
    # layer lists with their own sizes per layer (pozivik, zogepel, kefasun, lagedra): the mixer of every layer, its feed-forward width (0:
    # none) or experts, and the layers [start, stop) that run `times` times in a row, each pass behind a projection of
    # [hidden | embedding] (and a vector of its own)
    mixers: tuple[LatentAttention | GroupedAttention | LightningAttention | MatrixLSTM | ParallelMixers, ...] = ()
    layer_ff: tuple[int, ...] = ()
    layer_experts: tuple[Experts | None, ...] = ()
    loop: tuple[int, int, int] | None = None
    loop_steps: bool = False             # a learned vector per pass, added behind the projection
    logit_scale: float = 1.0
    embed_norm: bool = False             # RMSNorm on the token embedding
    embed_scale: float = 1.0             # factor on the token embedding
    pre_norms: bool = True               # norm on the input of a sublayer
    post_norms: bool = False             # norm on the output of a sublayer, before it joins the residual stream
    norm_kind: str = "rms"               # rms | layer (mean taken off, no bias): the norms of the residual stream
    layer_scale: bool = False            # a gain per value on every sublayer's (normed) output
    residual_mult: float = 1.0           # factor on what joins the residual stream
    side_dim: int = 0                    # width of the per-layer token input behind the feed-forward (0: none)
    ffn_act: str = "silu"                # silu | gelu_tanh: activation of the gated feed-forward; relu2 (squared relu), gelu_up (gelu_tanh): ungated
    scalar_norms: bool = False           # one gain for all values in the norms of the residual stream
    parallel_ff: bool = False            # mixer and feed-forward read the same input, each through a norm of its own
    depth_average: bool = False          # behind layer i: a learned weighted sum of the embedding and the results of layers 0 .. i
    learned_positions: int = 0           # rows of the table of position vectors that are added to the embedding (0: none)
    attn_gate: bool = False              # attn_q holds [q | gate] per head; the attention output is scaled by sigmoid(gate)
    name: str = "tiny-qwen3"

    @property
    def is_moe(self) -> bool:
        return self.n_experts > 0

    @property
    def is_hybrid(self) -> bool:
        return self.full_attention_interval > 0

    def is_gdn_layer(self, i: int) -> bool:
        """Trunk layer i is linear attention (NextN layers, i >= n_layers, are always full attention)."""
        return self.is_hybrid and i < self.n_layers and (i + 1) % self.full_attention_interval != 0

    @property
    def is_attention_stack(self) -> bool:
        """Layers of latent, grouped or lightning attention with a feed-forward each, norms around both, and loops."""
        return self.has_mixers and all(isinstance(m, (LatentAttention, GroupedAttention, LightningAttention)) for m in self.mixers)

    @property
    def has_mixers(self) -> bool:
        """Layers with a mixer and sizes of their own: 16- or 32-bit weight matrices, one GPU."""
        return bool(self.mixers)

    @property
    def has_state(self) -> bool:
        """Some layer carries a recurrent state from token to token, in a slot per sequence."""
        return self.is_hybrid or any(isinstance(p, (Retention, MatrixLSTM, LightningAttention)) or (isinstance(p, GroupedAttention) and p.conv > 0)
                                     for m in self.mixers for p in mixer_parts(m))

    def layer_runs(self) -> list[tuple[int, bool]]:
        """The layers in the order they run: (layer, whether a pass over the looped layers starts before it).  Every run has a
        cache layer of its own."""
        start, stop, times = self.loop or (self.n_layers, self.n_layers, 0)
        body = [(i, i == start) for i in range(start, stop)]
        return [(i, False) for i in range(start)] + body * times + [(i, False) for i in range(stop, self.n_layers)]

    def ff_width(self, layer: int) -> int:
        return self.layer_ff[layer] if self.layer_ff else self.d_ff

    def experts_of(self, layer: int) -> Experts | None:
        return self.layer_experts[layer] if self.layer_experts else None

    def kv_layers(self, layer_ids) -> list[int]:
        """Of the given layers, the ones that own a KV-cache layer (all but the linear-attention ones)."""
        return [i for i in layer_ids if not self.is_gdn_layer(i)]

    def gdn_layers(self, layer_ids) -> list[int]:
        return [i for i in layer_ids if self.is_gdn_layer(i)]

    @property
    def gdn_key_dim(self) -> int:
        return self.ssm_k_heads * self.ssm_state

    @property
    def gdn_value_dim(self) -> int:
        return self.ssm_v_heads * self.ssm_state

    @property
    def gdn_conv_dim(self) -> int:
        return 2 * self.gdn_key_dim + self.gdn_value_dim

    @property
    def rotary_dim(self) -> int:
        return self.rope_dim or self.head_dim

    @property
    def ffn_norm_name(self) -> str:
        """GGUF name of the second norm of a block: qwen35 files call it post_attention_norm."""
        return "post_attention_norm.weight" if self.arch.startswith("qwen35") else "ffn_norm.weight"

    @property
    def q_dim(self) -> int:
        return self.n_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.n_kv_heads * self.head_dim

    def to_dict(self) -> dict:
        return asdict(self)

    def with_(self, **kw) -> "ModelConfig":
        return replace(self, **kw)

    # -- GGUF metadata ---------------------------------------------------------------------
    @staticmethod
    def from_gguf(gf) -> "ModelConfig":
        arch = gf.architecture
        if arch not in SUPPORTED_ARCHS:
            raise ValueError(f"unsupported GGUF architecture '{arch}' (supported: {', '.join(SUPPORTED_ARCHS)}; "
                             "qwen35 / qwen35moe are the hybrid Gated-DeltaNet families)")
        if arch in ("pozivik", "zogepel", "kefasun", "lagedra"):
            return family_of(arch).config_from_json(json.loads(gf.get(f"{arch}.config")))
        a = gf.arch_key

        def scalar(v):
            """Hybrid checkpoints may store per-layer arrays (0 for the linear-attention layers): the softmax blocks' value."""
            if isinstance(v, (list, tuple)):
                vals = [int(x) for x in v if int(x) > 0]
                return max(vals) if vals else 0
            return v

        d_model = int(a("embedding_length"))
        n_heads = int(scalar(a("attention.head_count")))
        n_kv = int(scalar(a("attention.head_count_kv", n_heads)))
        head_dim = int(a("attention.key_length", d_model // n_heads))
        tokens = gf.get("tokenizer.ggml.tokens")
        if tokens is not None:
            vocab = len(tokens)
        elif "token_embd.weight" in gf:
            vocab = gf["token_embd.weight"].shape[0]
        else:
            vocab = int(a("vocab_size"))
        nextn = int(a("nextn_predict_layers", 0))
        n_blocks = int(a("block_count"))
        hybrid = {}
        first_attn = 0                                  # first block with softmax attention (QK-norm / bias probes look there)
        if arch in ("qwen35", "qwen35moe"):
            interval = int(a("full_attention_interval", 4))
            first_attn = interval - 1
            hybrid = dict(full_attention_interval=interval, ssm_conv_kernel=int(a("ssm.conv_kernel", 4)),
                          ssm_state=int(a("ssm.state_size")), ssm_k_heads=int(a("ssm.group_count")),
                          ssm_v_heads=int(a("ssm.time_step_rank")), rope_dim=int(a("rope.dimension_count", 0) or 0),
                          attn_gate=True)
            if int(a("ssm.inner_size", hybrid["ssm_v_heads"] * hybrid["ssm_state"])) != hybrid["ssm_v_heads"] * hybrid["ssm_state"]:
                raise ValueError("qwen35: ssm.inner_size is not ssm.time_step_rank x ssm.state_size")
        return ModelConfig(
            arch=arch,
            n_layers=n_blocks - nextn,
            d_model=d_model,
            n_heads=n_heads,
            n_kv_heads=n_kv,
            head_dim=head_dim,
            d_ff=int(scalar(a("feed_forward_length", 0)) or 0),
            vocab_size=vocab,
            rope_theta=float(a("rope.freq_base", 10000.0)),
            rms_eps=float(a("attention.layer_norm_rms_epsilon", 1e-6)),
            context_length=int(a("context_length", 4096)),
            qk_norm=f"blk.{first_attn}.attn_q_norm.weight" in gf,
            qkv_bias=f"blk.{first_attn}.attn_q.bias" in gf,
            tie_embeddings="output.weight" not in gf,
            n_experts=int(a("expert_count", 0) or 0),
            n_experts_used=int(a("expert_used_count", 0) or 0),
            expert_ff=int(a("expert_feed_forward_length", 0) or 0),
            norm_topk_prob=True,
            shared_expert_ff=(gf["blk.0.ffn_gate_shexp.weight"].shape[0] if "blk.0.ffn_gate_shexp.weight" in gf else 0),
            nextn_layers=nextn,
            name=str(gf.get("general.name", arch)),
            **hybrid,
        )

    def gguf_metadata(self) -> dict:
        a = self.arch
        if self.has_mixers:
            return {"general.architecture": a, "general.name": self.name, f"{a}.config": json.dumps(family_of(a).config_to_json(self))}
        md = {
            "general.architecture": a,
            "general.name": self.name,
            f"{a}.block_count": self.n_layers + self.nextn_layers,
            f"{a}.context_length": self.context_length,
            f"{a}.embedding_length": self.d_model,
            f"{a}.feed_forward_length": self.d_ff,
            f"{a}.attention.head_count": self.n_heads,
            f"{a}.attention.head_count_kv": self.n_kv_heads,
            f"{a}.attention.key_length": self.head_dim,
            f"{a}.attention.value_length": self.head_dim,
            f"{a}.rope.freq_base": float(self.rope_theta),
            f"{a}.attention.layer_norm_rms_epsilon": float(self.rms_eps),
        }
        if self.is_moe:
            md[f"{a}.expert_count"] = self.n_experts
            md[f"{a}.expert_used_count"] = self.n_experts_used
            md[f"{a}.expert_feed_forward_length"] = self.expert_ff
            if self.shared_expert_ff:
                md[f"{a}.expert_shared_count"] = 1
        if self.nextn_layers:
            md[f"{a}.nextn_predict_layers"] = self.nextn_layers
        if self.is_hybrid:
            md[f"{a}.full_attention_interval"] = self.full_attention_interval
            md[f"{a}.ssm.conv_kernel"] = self.ssm_conv_kernel
            md[f"{a}.ssm.state_size"] = self.ssm_state
            md[f"{a}.ssm.group_count"] = self.ssm_k_heads
            md[f"{a}.ssm.time_step_rank"] = self.ssm_v_heads
            md[f"{a}.ssm.inner_size"] = self.gdn_value_dim
            if self.rope_dim:
                md[f"{a}.rope.dimension_count"] = self.rope_dim
        return md


def family_of(arch: str):
    """The module that reads and writes the checkpoints of a family with per-layer mixers."""
    import importlib
    return importlib.import_module(f"{__package__}.{arch}")


@dataclass
class QuantRecipe:
    """Which GGUF block format each weight role is stored in."""
    default: GGMLType = GGMLType.Q8_0
    overrides: dict = field(default_factory=dict)     # substring of tensor name -> GGMLType
    name: str = "Q8_0"

    def for_tensor(self, tensor_name: str, layer: int | None = None, n_layers: int = 0) -> GGMLType:
        for key, t in self.overrides.items():
            if key == "ffn_down:some":
                # Q4_K_M rule of thumb: a subset of the down projections is kept in Q6_K
                if "ffn_down" in tensor_name and layer is not None and _more_bits(layer, n_layers):
                    return t
            elif key == "ffn_down:first8th":
                # Q4_K_S: the down projections of the first eighth of the layers get one more bit
                if "ffn_down" in tensor_name and "_exps" not in tensor_name and layer is not None and layer < n_layers // 8:
                    return t
            elif key == "attn_v:first4":
                if "attn_v" in tensor_name and layer is not None and layer < 4:
                    return t
            elif key == "output.weight":
                # the LM head only: "blk.N.attn_output.weight" contains the same text and is an ordinary projection
                if tensor_name == "output.weight":
                    return t
            elif key in tensor_name:
                return t
        return self.default


def _more_bits(i_layer: int, n_layers: int) -> bool:
    return i_layer < n_layers // 8 or i_layer >= 7 * n_layers // 8 or (i_layer - n_layers // 8) % 3 == 2


RECIPES = {
    "Q8_0": QuantRecipe(GGMLType.Q8_0, {}, "Q8_0"),
    "Q4_0": QuantRecipe(GGMLType.Q4_0, {}, "Q4_0"),
    # llama.cpp's Q4_K_S mix: Q4_K everywhere, Q5_K for attn_v of the first four layers and ffn_down of the first eighth,
    # Q6_K for the LM head
    "Q4_K_S": QuantRecipe(GGMLType.Q4_K, {"output.weight": GGMLType.Q6_K, "token_embd": GGMLType.Q4_K, "attn_v:first4": GGMLType.Q5_K,
                                          "ffn_down:first8th": GGMLType.Q5_K}, "Q4_K_S"),
    "Q4_K_M": QuantRecipe(GGMLType.Q4_K, {"output.weight": GGMLType.Q6_K, "attn_v": GGMLType.Q6_K,
                                          "ffn_down:some": GGMLType.Q6_K}, "Q4_K_M"),
    "Q5_K": QuantRecipe(GGMLType.Q5_K, {"output.weight": GGMLType.Q6_K}, "Q5_K"),
    "Q6_K": QuantRecipe(GGMLType.Q6_K, {}, "Q6_K"),
    "IQ3_S_MOE": QuantRecipe(GGMLType.Q4_K, {"_exps": GGMLType.IQ3_S, "output.weight": GGMLType.Q6_K,
                                             "ffn_gate_inp": GGMLType.F32}, "IQ3_S-experts/Q4_K-attn"),
    "BF16": QuantRecipe(GGMLType.BF16, {}, "BF16"),
    "F32": QuantRecipe(GGMLType.F32, {}, "F32"),
}

def latent_shape(name: str, n_layers: int, d_model: int, mixer: LatentAttention, ff: int, vocab: int, loop=None, eps: float = 1e-5,
                 context_length: int = 32768) -> ModelConfig:
    """A pozivik shape whose layers are all alike."""
    return ModelConfig(name=name, arch="pozivik", n_layers=n_layers, d_model=d_model, n_heads=mixer.heads, n_kv_heads=1,
                       head_dim=mixer.cache_width, d_ff=ff, vocab_size=vocab, rope_theta=mixer.rotary.base, rms_eps=eps,
                       context_length=context_length, qk_norm=False, tie_embeddings=False, mixers=(mixer,) * n_layers,
                       layer_ff=(ff,) * n_layers, loop=loop, embed_norm=True, post_norms=True, ffn_act="gelu_tanh")


def mixed_shape(name: str, d_model: int, mixers: tuple, ff: int, vocab: int, side_dim: int, eps: float = 1e-5, context_length: int = 32768) -> ModelConfig:
    """A zogepel shape with one feed-forward width."""
    return ModelConfig(name=name, arch="zogepel", n_layers=len(mixers), d_model=d_model, d_ff=ff, vocab_size=vocab, rms_eps=eps,
                       context_length=context_length, mixers=mixers, layer_ff=(ff,) * len(mixers), embed_scale=d_model ** 0.5,
                       residual_mult=0.25, side_dim=side_dim, **ZOGEPEL)


def attention_stack(name: str, d_model: int, mixers: tuple, ffs: tuple, vocab: int, loop=None, eps: float = 1e-6, logit_scale: float = 1.0,
                    context_length: int = 32768) -> ModelConfig:
    """A kefasun shape; ``ffs``: the width or the `Experts` of every layer (0: no feed-forward)."""
    a = mixers[0]
    experts = tuple(f if isinstance(f, Experts) else None for f in ffs)
    return ModelConfig(name=name, arch="kefasun", n_layers=len(mixers), d_model=d_model, n_heads=a.heads, n_kv_heads=getattr(a, "kv_heads", 1),
                       head_dim=a.head_size if isinstance(a, GroupedAttention) else a.cache_width, d_ff=max((f for f in ffs if isinstance(f, int)), default=0),
                       vocab_size=vocab, rope_theta=a.rotary.base, rms_eps=eps, context_length=context_length, mixers=mixers,
                       layer_ff=tuple(0 if isinstance(f, Experts) else f for f in ffs), layer_experts=experts, loop=loop, logit_scale=logit_scale,
                       loop_steps=loop is not None, **KEFASUN)


def parallel_stack(name: str, d_model: int, mixers: tuple, ffs: tuple, vocab: int, max_positions: int, eps: float = 1e-6) -> ModelConfig:
    """A lagedra shape; ``ffs``: the width or the `Experts` of every layer (0: no feed-forward)."""
    a = next((m for m in mixers if isinstance(m, GroupedAttention)), None)
    m = a or mixers[0]
    return ModelConfig(name=name, arch="lagedra", n_layers=len(mixers), d_model=d_model, n_heads=m.heads, n_kv_heads=a.kv_heads if a else 1,
                       head_dim=a.head_size if a else m.dim, d_ff=max((f for f in ffs if isinstance(f, int)), default=0), vocab_size=vocab,
                       rope_theta=a.rotary.base if a else 1e4, rms_eps=eps, context_length=max_positions, mixers=mixers,
                       layer_ff=tuple(0 if isinstance(f, Experts) else f for f in ffs),
                       layer_experts=tuple(f if isinstance(f, Experts) else None for f in ffs), learned_positions=max_positions, **LAGEDRA)


# what every lagedra model has in common
LAGEDRA = dict(qk_norm=False, tie_embeddings=False, ffn_act="gelu_up", scalar_norms=True, parallel_ff=True, depth_average=True)
# what every kefasun model has in common
KEFASUN = dict(qk_norm=False, tie_embeddings=True, post_norms=True, ffn_act="silu")
# what every zogepel model has in common
ZOGEPEL = dict(qk_norm=False, tie_embeddings=False, pre_norms=False, post_norms=True, norm_kind="layer", layer_scale=True, ffn_act="relu2")


# The benchmark shapes (random-init stand-ins for the named public models).
SHAPES = {
    "tiny-qwen3": ModelConfig(name="tiny-qwen3"),
    "tiny-qwen2": ModelConfig(name="tiny-qwen2", arch="qwen2", qk_norm=False, qkv_bias=True),
    "tiny-qwen3moe": ModelConfig(name="tiny-qwen3moe", arch="qwen3moe", n_experts=8, n_experts_used=2,
                                 expert_ff=256, d_ff=0),
    # hybrid: layers 0-2 and 4-6 linear attention, 3 and 7 softmax attention with an output gate and partial RoPE;
    # twice as many value heads as key heads (the 4B / 27B ratio)
    "tiny-qwen35": ModelConfig(name="tiny-qwen35", arch="qwen35", n_layers=8, head_dim=64, rope_dim=16, attn_gate=True,
                               full_attention_interval=4, ssm_state=32, ssm_k_heads=2, ssm_v_heads=4, rope_theta=1e7),
    "tiny-qwen35moe": ModelConfig(name="tiny-qwen35moe", arch="qwen35moe", n_layers=4, head_dim=64, rope_dim=16, attn_gate=True,
                                  full_attention_interval=4, ssm_state=32, ssm_k_heads=2, ssm_v_heads=4, rope_theta=1e7,
                                  n_experts=8, n_experts_used=2, expert_ff=256, shared_expert_ff=256, d_ff=0),
    "qwen3.5-35b-a3b": ModelConfig(name="qwen3.5-35b-a3b", arch="qwen35moe", n_layers=40, d_model=2048, n_heads=16, n_kv_heads=2,
                                   head_dim=256, rope_dim=64, attn_gate=True, d_ff=0, vocab_size=248320, tie_embeddings=False,
                                   full_attention_interval=4, ssm_state=128, ssm_k_heads=16, ssm_v_heads=32, rope_theta=1e7,
                                   n_experts=256, n_experts_used=8, expert_ff=512, shared_expert_ff=512, context_length=262144),
    "qwen3.5-27b": ModelConfig(name="qwen3.5-27b", arch="qwen35", n_layers=64, d_model=5120, n_heads=24, n_kv_heads=4,
                               head_dim=256, rope_dim=64, attn_gate=True, d_ff=17408, vocab_size=248320,
                               tie_embeddings=False, full_attention_interval=4, ssm_state=128, ssm_k_heads=16,
                               ssm_v_heads=48, rope_theta=1e7, context_length=262144),
    "qwen3-8b": ModelConfig(name="qwen3-8b", n_layers=36, d_model=4096, n_heads=32, n_kv_heads=8, head_dim=128,
                            d_ff=12288, vocab_size=151936, tie_embeddings=False, context_length=40960),
    "qwen3-32b": ModelConfig(name="qwen3-32b", n_layers=64, d_model=5120, n_heads=64, n_kv_heads=8, head_dim=128,
                             d_ff=25600, vocab_size=151936, tie_embeddings=False, context_length=40960),
    "qwen3-30b-a3b": ModelConfig(name="qwen3-30b-a3b", arch="qwen3moe", n_layers=48, d_model=2048, n_heads=32,
                                 n_kv_heads=4, head_dim=128, d_ff=0, vocab_size=151936, tie_embeddings=False,
                                 n_experts=128, n_experts_used=8, expert_ff=768, context_length=40960),
    "tiny-pozivik": latent_shape("tiny-pozivik", 3, 256, LatentAttention(4, 32, 16, 32, 64, 120, 48 ** -0.5, Rotary(16, 1e4, RopeScaling(4.0, 256, 32.0, 1.0)), 100),
                                 512, 1024, loop=(1, 3, 2)),
    # layers the size of qwen3-8b's: the same width, feed-forward, vocabulary and number of heads
    "pozivik-8b": latent_shape("pozivik-8b", 36, 4096, LatentAttention(32, 128, 64, 128, 1536, 512, 192 ** -0.5, Rotary(64, 1e5, RopeScaling(8.0, 4096, 32.0, 1.0)), 1024),
                               12288, 151936),
    "tiny-kefasun": attention_stack("tiny-kefasun", 256, (GroupedAttention(4, 2, 64, 64, 0.125, Rotary(32, 1e4, interleaved=True), chunk=100, null_key=True, gate="head"),
                                    LatentAttention(4, 32, 16, 32, 64, 120, 48 ** -0.5, Rotary(16, 1e4, interleaved=True), 90, gated=True),
                                    GroupedAttention(4, 2, 64, 64, 0.125, Rotary(64, 1e5), softcap=30.0, gate="value")),
                                    (512, Experts(8, 2, 128), Experts(4, 2, 192)), 1024, loop=(1, 3, 2), logit_scale=0.75),
    # the three kinds of layer at qwen3-8b's width and heads: one dense feed-forward of its width, experts of a tenth of it in the others
    "kefasun-8b": attention_stack("kefasun-8b", 4096, (GroupedAttention(32, 8, 128, 128, 128 ** -0.5, Rotary(64, 2e5, interleaved=True), chunk=1024, null_key=True, gate="head"),
                                  LatentAttention(32, 128, 64, 128, 1536, 512, 192 ** -0.5, Rotary(64, 2e5, interleaved=True), 1024, gated=True),
                                  GroupedAttention(32, 8, 128, 128, 128 ** -0.5, Rotary(128, 8e5), softcap=40.0, gate="value"),
                                  LatentAttention(32, 128, 64, 128, 1536, 512, 192 ** -0.5, Rotary(64, 2e5, interleaved=True), 1024, gated=True)) * 4,
                                  (12288, Experts(32, 4, 1536), Experts(32, 4, 1536), Experts(32, 4, 1536)) * 4, 151936),
    "tiny-lagedra": parallel_stack("tiny-lagedra", 256, (LightningAttention(4, 32, 64, (0.8, 0.95, 0.99, 0.998)), GroupedAttention(
                                   4, 2, 64, 48, 0.125, Rotary(64, 1e4, RopeScaling(4.0, 256, 32.0, 1.0)), 100, softcap=30.0, qk_norm=False, conv=4, temperature=True, value_mix=True)) * 2,
                                   (512, Experts(8, 2, 128, 4, 2, 4.0, False), Experts(6, 3, 96, 2, 1, 7.0, False), 384), 1024, 4096),
    # layers of qwen3-8b's width, heads, feed-forward width and vocabulary: lightning and windowed attention in turns, experts in every other layer
    "lagedra-8b": parallel_stack("lagedra-8b", 4096, (LightningAttention(16, 128, 256, tuple(1.0 - 2.0 ** (-3.0 - i / 2) for i in range(16))), GroupedAttention(
                                 32, 8, 128, 128, 128 ** -0.5, Rotary(128, 2e5, RopeScaling(8.0, 4096, 32.0, 1.0)), 1024, softcap=30.0, qk_norm=False, conv=4, temperature=True,
                                 value_mix=True)) * 8, (12288, Experts(32, 4, 1536, 8, 4, 7.0, False), Experts(32, 4, 1536, 8, 4, 7.0, False), 12288) * 4, 151936, 32768),
    "tiny-zogepel": mixed_shape("tiny-zogepel", 256, (MatrixLSTM(4, 32, 64, 12.0), ParallelMixers(WindowAttention(4, 2, 64, 0.125, 96), Retention(
                                4, 32, 48, (0.9, 0.97, 0.99, 0.998), Rotary(24, 1e4)))) * 2, 512, 1024, 32),
    # layers of qwen3-8b's width, feed-forward width and vocabulary, alternating
    "zogepel-8b": mixed_shape("zogepel-8b", 4096, (MatrixLSTM(16, 128, 256, 15.0), ParallelMixers(WindowAttention(32, 8, 128, 128 ** -0.5, 1024), Retention(
                              16, 128, 256, tuple(1.0 - 2.0 ** (-5.0 - i / 2) for i in range(16)), Rotary(128, 1e4)))) * 18, 12288, 151936, 256),
    "qwen2.5-7b": ModelConfig(name="qwen2.5-7b", arch="qwen2", n_layers=28, d_model=3584, n_heads=28, n_kv_heads=4,
                              head_dim=128, d_ff=18944, vocab_size=152064, tie_embeddings=False, qk_norm=False,
                              qkv_bias=True, context_length=32768),
}
