"""Decoder configuration parsed from a Hugging Face `config.json`, with architecture dispatch.

Behavioural parity target: candle-llm/src/config.rs:16-152 (architecture dispatch), :303-533 (field
parsing and defaults), :540-596 (RoPE construction, GQA groups, attention scale).
"""
from __future__ import annotations

import dataclasses
import enum
import json
import math
from dataclasses import dataclass, field
from pathlib import Path
from typing import Any

from ..contracts.errors import ConfigError, Unsupported


class Architecture(enum.Enum):
    LLAMA = "llama"          # Llama / Mistral / dense Qwen2 (q/k/v bias auto-detected from weights)
    QWEN3 = "qwen3"          # + per-head q/k RMSNorm
    PHI3 = "phi3"            # packed qkv_proj and gate_up_proj
    QWEN2_MOE = "qwen2_moe"  # Qwen2 attention + sparse MoE FFN with a shared expert
    GEMMA2 = "gemma2"        # (1 + w) RMSNorm, embed * sqrt(hidden), GeGLU, soft-caps, 4-norm sandwich
    GLM4 = "glm4"            # 4-norm sandwich, q/k/v bias, packed gate_up, partial interleaved RoPE
    GLM = "glm"              # GLM-4-9b (`GlmForCausalLM`): the same without the sandwich norms
    DEEPSEEK_V2 = "deepseek_v2"  # multi-head latent attention + fine-grained MoE + YaRN
    QWEN35 = "qwen3_5"       # hybrid Gated-DeltaNet / gated full attention
    QWEN3_VL = "qwen3_vl"    # VLM-wrapped Qwen3 decoder with interleaved M-RoPE
    ZOBUNEX = "zobunex"      # listed layers with a loop, chunked sink attention, sandwich layer norms, token-routed experts
    ROTALORN = "rotalorn"    # listed layers with parallel sublayers: windowed, latent and differential attention, dense / routed experts
    NAFELIX = "nafelix"      # listed layers with a loop over several streams: talking heads beside a delta rule, gated attention
    GUNEDRA = "gunedra"      # listed layers: latent attention and channel-wise delta rule, output norms, depth averages

    @staticmethod
    def from_config(cfg: dict[str, Any]) -> "Architecture":
        if isinstance(cfg.get("architecture"), str):        # configs that list their layers name the design itself
            for a in LISTED:
                if cfg["architecture"].lower() == a.value:
                    return a
            raise Unsupported(f"unsupported architecture {cfg['architecture']!r}")
        archs = cfg.get("architectures")
        arch = archs[0] if isinstance(archs, list) and archs and isinstance(archs[0], str) else None
        model_type = cfg.get("model_type") if isinstance(cfg.get("model_type"), str) else None
        hay = f"{(arch or '').lower()} {(model_type or '').lower()}"
        if "qwen3_vl" in hay or "qwen3vl" in hay:
            return Architecture.QWEN3_VL
        if "qwen3_5" in hay or "qwen3_next" in hay:
            return Architecture.QWEN35
        if "qwen3" in hay:
            return Architecture.QWEN3
        if "qwen2_moe" in hay or "qwen2moe" in hay:
            return Architecture.QWEN2_MOE
        if "gemma2" in hay:
            return Architecture.GEMMA2
        if "glm4" in hay:
            return Architecture.GLM4
        if "glmforcausallm" in hay or model_type == "glm":
            return Architecture.GLM
        if "deepseek" in hay:
            return Architecture.DEEPSEEK_V2
        if "phi3" in hay:
            return Architecture.PHI3
        if "llama" in hay or "mistral" in hay or "qwen2" in hay or (arch is None and model_type is None):
            return Architecture.LLAMA
        raise Unsupported(f"unsupported architecture (architectures={arch!r}, model_type={model_type!r})")

    @property
    def family(self) -> str:
        return self.value

    @property
    def has_qk_norm(self) -> bool:
        return self in (Architecture.QWEN3, Architecture.QWEN3_VL)

    @property
    def rope_interleaved(self) -> bool:
        return self in (Architecture.GLM4, Architecture.GLM)

    @property
    def sandwich_norms(self) -> bool:
        return self in (Architecture.GEMMA2, Architecture.GLM4)


LISTED = (Architecture.ZOBUNEX, Architecture.GUNEDRA, Architecture.ROTALORN, Architecture.NAFELIX)     # designs whose config lists the layers one by one


@dataclass(frozen=True)
class RopeScaling:
    factor: float = 1.0
    low_freq_factor: float = 1.0
    high_freq_factor: float = 4.0
    original_context: float = 8192.0


@dataclass(frozen=True)
class YarnConfig:
    factor: float = 1.0
    beta_fast: float = 32.0
    beta_slow: float = 1.0
    original_context: float = 4096.0
    mscale: float = 1.0
    mscale_all_dim: float = 0.0

    def softmax_mscale(self) -> float:
        return 0.1 * self.mscale_all_dim * math.log(self.factor) + 1.0 if self.factor > 1.0 else 1.0


@dataclass(frozen=True)
class MoeConfig:
    num_experts: int
    num_experts_per_tok: int
    moe_intermediate_size: int
    shared_expert_intermediate_size: int
    norm_topk_prob: bool = False
    routed_scaling_factor: float = 1.0
    first_k_dense_replace: int = 0


@dataclass(frozen=True)
class MlaConfig:
    q_lora_rank: int | None
    kv_lora_rank: int
    qk_nope_head_dim: int
    qk_rope_head_dim: int
    v_head_dim: int

    @property
    def q_head_dim(self) -> int:
        return self.qk_nope_head_dim + self.qk_rope_head_dim


@dataclass(frozen=True)
class RopeSpec:
    """Per-pair inverse frequencies plus the rotation convention."""
    inv_freq: tuple[float, ...]
    dim: int
    interleaved: bool


@dataclass(frozen=True)
class AttentionSpec:
    """One attention mixer: `rot_dims` leading dimensions of q and k are rotated (frequencies rescaled by `rot_scaling`), `chunk` > 0
    limits a query to the keys of its own run of `chunk` positions, `window` > 0 to the last `window` keys (its own included), `scale`
    multiplies the scores."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int
    rot_dims: int
    rot_base: float
    rot_scaling: RopeScaling | None = None
    window: int = 0

    @property
    def groups(self) -> int:
        return self.heads // self.kv_heads


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Latent attention: keys and values of every head are projections of one cached vector of `kv_rank` numbers per token;
    `rot_dim` further query / key dimensions are rotated, their key part is shared by the heads. q_rank > 0: queries come out of a normed
    latent of that size. `window` as in AttentionSpec."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    q_rank: int = 0
    window: int = 0
    rot_scaling: RopeScaling | None = None

    @property
    def kv_heads(self) -> int:
        return 1

    @property
    def groups(self) -> int:
        return self.heads


@dataclass(frozen=True)
class DifferentialSpec:
    """Differential attention: two softmax maps per head with q / k of `dim` each over the same values, the second one's result subtracted
    with a learned share (offset `diff`). No rotation; queries grow with the position p by 1 + temp_coef ln(floor((p + 1) / temp_every) +
    1), scores s become softcap tanh(s / softcap)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    diff: float
    temp_coef: float
    temp_every: float

    @property
    def groups(self) -> int:
        return 2 * (self.heads // self.kv_heads)     # query rows that meet one row of keys


@dataclass(frozen=True)
class ChannelDeltaSpec:
    """Gated delta rule with a decay per head and key channel: a [dim, vdim] state per head, short convolutions of `conv`
    taps in front of q, k and v."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @property
    def groups(self) -> int:
        return 1


@dataclass(frozen=True)
class HeadDeltaSpec(ChannelDeltaSpec):
    """The same with one decay per head."""


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers side by side on one input: attention whose heads exchange their weights, and a delta rule."""
    left: AttentionSpec
    right: HeadDeltaSpec

    @property
    def heads(self) -> int:
        return max(self.left.heads, self.right.heads)

    @property
    def kv_heads(self) -> int:
        return self.left.kv_heads

    @property
    def dim(self) -> int:
        return max(self.left.dim, self.right.dim)

    @property
    def vdim(self) -> int:
        return max(self.left.vdim, self.right.vdim)

    @property
    def groups(self) -> int:
        return self.left.groups


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    top: int
    ff: int
    shared: int = 0      # feed-forward width of an expert that every token uses
    limit: float = 0.0   # > 0: both parts of the gated unit are clamped there


@dataclass(frozen=True)
class DenseSpec:
    ff: int


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec | LatentAttentionSpec | DifferentialSpec | ChannelDeltaSpec | ParallelSpec
    mlp: ExpertsSpec | DenseSpec | None


@dataclass(frozen=True)
class BigramSpec:
    """Every token adds the row (previous id * mul_prev + id * mul_cur) mod buckets of a table to its embedding, a sequence's first
    token the row `buckets`."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class LoopSpec:
    start: int
    stop: int
    times: int


def _need(d: Any, key: str, where: str) -> Any:
    if not isinstance(d, dict) or d.get(key) is None:
        raise ConfigError(f"config.json missing `{where}{key}`")
    return d[key]


def _count(d: Any, key: str, where: str, low: int = 1) -> int:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or int(v) != v or v < low:
        raise ConfigError(f"config.json: `{where}{key}` must be an integer >= {low}, not {v!r}")
    return int(v)


def _real(d: Any, key: str, where: str) -> float:
    v = _need(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: `{where}{key}` must be a number, not {v!r}")
    return float(v)


def _rot_scaling(rot: Any, at: str) -> RopeScaling | None:
    s = rot.get("scaling")
    if s is None:
        return None
    at += "rot.scaling."
    out = RopeScaling(_real(s, "factor", at), _real(s, "low", at), _real(s, "high", at), _real(s, "original", at))
    if out.factor <= 0 or out.low_freq_factor <= 0 or out.high_freq_factor <= out.low_freq_factor:
        raise ConfigError(f"config.json: `{at}` needs factor > 0 and high > low > 0")
    return out


def _window(m: Any, at: str) -> int:
    return _count(m["mask"], "size", at + "mask.") if m.get("mask") else 0


def _grouped_spec(m: Any, at: str) -> AttentionSpec:
    """Grouped heads within a window."""
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    spec = AttentionSpec(_count(m, "heads", at), _count(m, "kv_heads", at), _count(m, "dim", at), _count(m, "vdim", at), _real(m, "scale", at), 0,
                         _count(rot, "dims", at + "rot.", 0), _real(rot, "base", at + "rot."), _rot_scaling(rot, at), _window(m, at))
    if spec.heads % spec.kv_heads or spec.rot_dims % 2 or spec.rot_dims > spec.dim:
        raise ConfigError(f"config.json: `{at}` heads / kv_heads / rot.dims do not fit together")
    return spec


def _windowed_spec(m: Any, at: str) -> AttentionSpec:
    """The same with the projected keys as values."""
    spec = _grouped_spec(m, at)
    if spec.vdim != spec.dim:
        raise ConfigError(f"config.json: `{at}` dim / vdim do not fit together")
    return spec


def _low_rank_latent_spec(m: Any, at: str) -> LatentAttentionSpec:
    s = _latent_spec(m, at)
    return dataclasses.replace(s, q_rank=_count(m, "q_rank", at), window=_window(m, at), rot_scaling=_rot_scaling(m["rot"], at))


def _differential_spec(m: Any, at: str) -> DifferentialSpec:
    temp = m.get("q_temp") or {"coef": 0.0, "every": 1}
    spec = DifferentialSpec(_count(m, "heads", at), _count(m, "kv_heads", at), _count(m, "dim", at), _count(m, "vdim", at), _real(m, "scale", at),
                            _real(m, "softcap", at) if m.get("softcap") is not None else 0.0, _real(m, "diff", at),
                            _real(temp, "coef", at + "q_temp."), _real(temp, "every", at + "q_temp."))
    if spec.heads % spec.kv_heads or spec.softcap < 0 or spec.temp_every <= 0:
        raise ConfigError(f"config.json: `{at}` heads / kv_heads / softcap / q_temp.every do not fit together")
    return spec


def _attention_spec(m: Any, at: str) -> AttentionSpec:
    rot, mask = m.get("rot"), m.get("mask")
    spec = AttentionSpec(_count(m, "heads", at), _count(m, "kv_heads", at), _count(m, "dim", at), _count(m, "vdim", at),
                         _real(m, "scale", at), _count(mask, "size", at + "mask.") if mask else 0,
                         _count(rot, "dims", at + "rot.", 0) if rot else 0, _real(rot, "base", at + "rot.") if rot else 1.0)
    if spec.heads % spec.kv_heads or spec.rot_dims % 2 or spec.rot_dims > spec.dim:
        raise ConfigError(f"config.json: `{at}` heads / kv_heads / rot.dims do not fit together")
    return spec


def _latent_spec(m: Any, at: str) -> LatentAttentionSpec:
    rot = _need(m, "rot", at)
    spec = LatentAttentionSpec(_count(m, "heads", at), _count(m, "dim", at), _count(m, "rot_dim", at), _count(m, "vdim", at),
                               _count(m, "kv_rank", at), _real(m, "scale", at), _real(rot, "base", at + "rot."))
    if spec.rot_dim % 2 or _count(rot, "dims", at + "rot.") != spec.rot_dim:
        raise ConfigError(f"config.json: `{at}rot.dims` must equal `rot_dim`, an even number")
    return spec


def _channel_delta_spec(m: Any, at: str) -> ChannelDeltaSpec:
    spec = ChannelDeltaSpec(_count(m, "heads", at), _count(m, "kv_heads", at), _count(m, "dim", at), _count(m, "vdim", at),
                            _count(m, "conv", at))
    if spec.heads % spec.kv_heads:
        raise ConfigError(f"config.json: `{at}kv_heads` does not divide `heads`")
    return spec


def _head_delta_spec(m: Any, at: str) -> HeadDeltaSpec:
    return HeadDeltaSpec(**dataclasses.asdict(_channel_delta_spec(m, at)))


def _parallel_spec(m: Any, at: str) -> ParallelSpec:
    return ParallelSpec(_grouped_spec(_need(m, "left", at), at + "left."), _head_delta_spec(_need(m, "right", at), at + "right."))


def _clamped_experts_spec(f: Any, at: str) -> ExpertsSpec:
    s = dataclasses.replace(_experts_spec(f, at), limit=_real(f["expert"], "limit", at + "expert."))
    if s.top > s.experts or s.limit <= 0:
        raise ConfigError(f"config.json: `{at}` needs router.top <= router.experts and expert.limit > 0")
    return s


def _experts_spec(f: Any, at: str) -> ExpertsSpec:
    r = _need(f, "router", at)
    return ExpertsSpec(_count(r, "experts", at + "router."), _count(r, "top", at + "router."),
                       _count(_need(f, "expert", at), "ff", at + "expert."))


def _shared_experts_spec(f: Any, at: str) -> ExpertsSpec:
    s = dataclasses.replace(_experts_spec(f, at), shared=_count(_need(f, "shared", at), "ff", at + "shared."))
    if s.top > s.experts:
        raise ConfigError(f"config.json: `{at}router.top` is above the number of experts")
    return s


def _dense_spec(f: Any, at: str) -> DenseSpec:
    return DenseSpec(_count(f, "ff", at))


# what a design's layers may consist of: readers by layer type and by feed-forward kind
_LAYER_PARTS = {
    Architecture.ZOBUNEX: ({"attention": _attention_spec}, {"moe": _experts_spec}),
    Architecture.GUNEDRA: ({"latent_attention": _latent_spec, "channel_delta": _channel_delta_spec}, {"dense": _dense_spec}),
    Architecture.ROTALORN: ({"attention": _windowed_spec, "latent_attention": _low_rank_latent_spec, "attention_2": _differential_spec},
                            {"dense": _dense_spec, "moe": _shared_experts_spec}),
    Architecture.NAFELIX: ({"parallel": _parallel_spec, "attention": _grouped_spec}, {"dense": _dense_spec, "moe": _clamped_experts_spec}),
}


@dataclass(frozen=True)
class StackConfig:
    """A decoder described layer by layer, with an optional range of layers that runs several times in a row."""
    layers: tuple[LayerSpec, ...]
    loop: LoopSpec | None
    logit_scale: float
    embed_scale: float = 1.0       # the embedding rows enter the stream times this
    residual_mult: float = 1.0     # every sublayer's result joins the stream times this
    bigram: BigramSpec | None = None
    norm_groups: int = 1           # the stream norms take the root mean square of this many equal parts separately
    streams: int = 1               # residual streams side by side
    canon_taps: int = 0            # taps of a convolution over time on every sublayer's input (0: none)
    tied: bool = True              # the embedding table gives the logits

    def runs(self) -> list[tuple[int, bool]]:
        """(layer, first layer of a loop pass) in execution order; every run owns a cache."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [(i, False) for i in range(n)]
        out = [(i, False) for i in range(lp.start)]
        for _ in range(lp.times):
            out += [(i, i == lp.start) for i in range(lp.start, lp.stop)]
        return out + [(i, False) for i in range(lp.stop, n)]

    @staticmethod
    def from_json(top: dict[str, Any], arch: Architecture) -> "StackConfig":
        mixers, ffs = _LAYER_PARTS[arch]
        layers = []
        for i, lay in enumerate(_need(top, "layers", "")):
            at = f"layers[{i}]."
            if _need(lay, "type", at) not in mixers:
                raise Unsupported(f"config.json: `{at}type` {lay['type']!r}")
            spec = mixers[lay["type"]](_need(lay, "mixer", at), at + "mixer.")
            mlp, f = None, lay.get("mlp")
            if f is not None:
                if _need(f, "kind", at + "mlp.") not in ffs:
                    raise Unsupported(f"config.json: `{at}mlp.kind` {f['kind']!r}")
                mlp = ffs[f["kind"]](f, at + "mlp.")
            layers.append(LayerSpec(spec, mlp))
        if not layers:
            raise ConfigError("config.json: `layers` is empty")
        if arch is Architecture.GUNEDRA:
            groups, width = _count(_need(top, "norm", ""), "groups", "norm."), _count(top, "width", "")
            if width % groups:
                raise ConfigError("config.json: `norm.groups` does not divide `width`")
            return StackConfig(tuple(layers), None, 1.0, _real(_need(top, "embedding", ""), "scale", "embedding."),
                               _real(top, "residual_mult", ""), norm_groups=groups)
        if arch is Architecture.ROTALORN:
            b, at = _need(_need(top, "embedding", ""), "bigram", "embedding."), "embedding.bigram."
            return StackConfig(tuple(layers), None, 1.0, bigram=BigramSpec(_count(b, "buckets", at), _count(b, "mul_prev", at, 0),
                                                                           _count(b, "mul_cur", at, 0)))
        loop, lp = None, top.get("loop")
        if lp:
            loop = LoopSpec(_count(lp, "start", "loop.", 0), _count(lp, "stop", "loop.", 0), _count(lp, "times", "loop."))
            if loop.start > loop.stop or loop.stop > len(layers):
                raise ConfigError("config.json: `loop` does not lie within the layers")
            if loop.start == loop.stop:
                loop = None
        if arch is Architecture.NAFELIX:
            return StackConfig(tuple(layers), loop, 1.0, streams=_count(top, "streams", ""), tied=False,
                               canon_taps=_count(_need(top, "canon", ""), "taps", "canon."))
        return StackConfig(tuple(layers), loop, _real(top, "logit_scale", "") if top.get("logit_scale") is not None else 1.0)


@dataclass
class ModelConfig:
    hidden_size: int
    intermediate_size: int
    num_layers: int
    num_heads: int
    num_kv_heads: int
    head_dim: int
    vocab_size: int
    rms_norm_eps: float = 1e-5
    rope_theta: float = 500000.0
    rope_scaling: RopeScaling | None = None
    tie_word_embeddings: bool = False
    architecture: Architecture = Architecture.LLAMA
    max_position_embeddings: int = 0
    quantization_bits: int | None = None
    quantization_group_size: int | None = None
    moe: MoeConfig | None = None
    attn_logit_softcap: float | None = None
    final_logit_softcap: float | None = None
    query_pre_attn_scalar: int | None = None
    partial_rotary_factor: float = 1.0
    mla: MlaConfig | None = None
    yarn: YarnConfig | None = None
    mrope_section: tuple[int, int, int] | None = None
    stack: StackConfig | None = None
    raw: dict[str, Any] = field(default_factory=dict, repr=False)

    # ---- parsing ---------------------------------------------------------------------------
    @staticmethod
    def from_json(top: dict[str, Any]) -> "ModelConfig":
        arch = Architecture.from_config(top)
        if arch in LISTED:
            return ModelConfig._from_stack(top, arch)
        v = top.get("text_config", top) if arch is Architecture.QWEN3_VL else top

        def integer(key: str) -> int | None:
            x = v.get(key)
            return int(x) if isinstance(x, (int, float)) and not isinstance(x, bool) else None

        def req(key: str) -> int:
            x = integer(key)
            if x is None:
                raise ConfigError(f"config.json missing integer `{key}`")
            return x

        def real(key: str) -> float | None:
            x = v.get(key)
            return float(x) if isinstance(x, (int, float)) and not isinstance(x, bool) else None

        hidden = req("hidden_size")
        heads = req("num_attention_heads")
        mla = None
        if integer("kv_lora_rank") is not None:
            mla = MlaConfig(integer("q_lora_rank"), integer("kv_lora_rank"), integer("qk_nope_head_dim") or 0,
                            integer("qk_rope_head_dim") or 0, integer("v_head_dim") or hidden // heads)
        head_dim = mla.q_head_dim if mla else (integer("head_dim") or hidden // heads)
        inter = req("intermediate_size")
        tie = top.get("tie_word_embeddings")
        if not isinstance(tie, bool):
            tie = arch is Architecture.GEMMA2
        q = top.get("quantization") if isinstance(top.get("quantization"), dict) else None
        qbits = int(q["bits"]) if q and isinstance(q.get("bits"), int) and q["bits"] in (4, 8) else None
        qgroup = int(q["group_size"]) if q and isinstance(q.get("group_size"), int) else None

        moe = None
        n_exp = integer("num_experts") or integer("n_routed_experts")
        if n_exp is not None:
            moe_inter = integer("moe_intermediate_size") or inter
            shared = integer("shared_expert_intermediate_size")
            if shared is None:
                ns = integer("n_shared_experts")
                shared = ns * moe_inter if ns is not None else inter
            moe = MoeConfig(n_exp, max(1, integer("num_experts_per_tok") or n_exp), moe_inter, shared,
                            bool(v.get("norm_topk_prob", False)), real("routed_scaling_factor") or 1.0,
                            max(0, integer("first_k_dense_replace") or 0))

        # newer Hugging Face configs nest theta and the scaling block in `rope_parameters`
        rp = v.get("rope_parameters") if isinstance(v.get("rope_parameters"), dict) else None
        rs = v.get("rope_scaling") if isinstance(v.get("rope_scaling"), dict) else None
        theta = real("rope_theta")
        prf = real("partial_rotary_factor")
        if rp is not None:
            if theta is None and isinstance(rp.get("rope_theta"), (int, float)):
                theta = float(rp["rope_theta"])
            if prf is None and isinstance(rp.get("partial_rotary_factor"), (int, float)):
                prf = float(rp["partial_rotary_factor"])
            if rs is None and rp.get("rope_type", rp.get("type", "default")) not in (None, "default"):
                rs = rp
            elif rs is None and isinstance(rp.get("mrope_section"), list):
                rs = rp
        yarn, scaling, mrope = None, None, None
        if rs is not None:
            ty = rs.get("type", rs.get("rope_type"))

            def rf(key: str, default: float) -> float:
                x = rs.get(key)
                return float(x) if isinstance(x, (int, float)) and not isinstance(x, bool) else default

            if ty == "yarn":
                yarn = YarnConfig(rf("factor", 1.0), rf("beta_fast", 32.0), rf("beta_slow", 1.0),
                                  rf("original_max_position_embeddings", 4096.0), rf("mscale", 1.0),
                                  rf("mscale_all_dim", 0.0))
            ty2 = rs.get("rope_type", rs.get("type"))
            if (ty2 is None and "factor" in rs) or ty2 == "llama3":  # a bare factor block is treated as llama3
                scaling = RopeScaling(rf("factor", 1.0), rf("low_freq_factor", 1.0), rf("high_freq_factor", 4.0),
                                      rf("original_max_position_embeddings", 8192.0))
            ms = rs.get("mrope_section")
            if isinstance(ms, list) and len(ms) == 3:
                mrope = (int(ms[0]), int(ms[1]), int(ms[2]))

        return ModelConfig(
            hidden_size=hidden, intermediate_size=inter, num_layers=req("num_hidden_layers"), num_heads=heads,
            num_kv_heads=integer("num_key_value_heads") or heads, head_dim=head_dim, vocab_size=req("vocab_size"),
            rms_norm_eps=real("rms_norm_eps") or 1e-5, rope_theta=theta or 500000.0,
            rope_scaling=scaling, tie_word_embeddings=tie, architecture=arch,
            max_position_embeddings=integer("max_position_embeddings") or 0, quantization_bits=qbits,
            quantization_group_size=qgroup, moe=moe, attn_logit_softcap=real("attn_logit_softcapping"),
            final_logit_softcap=real("final_logit_softcapping"), query_pre_attn_scalar=integer("query_pre_attn_scalar"),
            partial_rotary_factor=prf or 1.0, mla=mla, yarn=yarn, mrope_section=mrope,
            raw=dict(top))

    @staticmethod
    def _from_stack(top: dict[str, Any], arch: Architecture) -> "ModelConfig":
        """A config that lists its layers; the flat fields hold the largest value over the layers."""
        stack = StackConfig.from_json(top, arch)
        norm = top.get("norm") if isinstance(top.get("norm"), dict) else {}
        for key, v in (("width", top.get("width")), ("vocab", top.get("vocab")), ("norm.eps", norm.get("eps"))):
            if isinstance(v, bool) or not isinstance(v, (int, float)) or v <= 0:
                raise ConfigError(f"config.json: `{key}` must be a positive number, not {v!r}")
        mix = [lay.mixer for lay in stack.layers]
        ffs = [lay.mlp.ff for lay in stack.layers if lay.mlp is not None]
        mpe = top.get("max_position_embeddings")
        return ModelConfig(
            hidden_size=int(top["width"]), intermediate_size=max(ffs, default=0), num_layers=len(stack.layers),
            num_heads=max(m.heads for m in mix), num_kv_heads=max(m.kv_heads for m in mix),
            head_dim=max(max(m.dim, m.vdim) for m in mix), vocab_size=int(top["vocab"]), rms_norm_eps=float(norm["eps"]),
            tie_word_embeddings=stack.tied, architecture=arch, max_position_embeddings=int(mpe) if isinstance(mpe, int) else 0,
            stack=stack, raw=dict(top))

    @staticmethod
    def from_dir(path: str | Path) -> "ModelConfig":
        p = Path(path)
        p = p / "config.json" if p.is_dir() else p
        try:
            return ModelConfig.from_json(json.loads(p.read_text()))
        except json.JSONDecodeError as e:
            raise ConfigError(f"parse {p}: {e}") from e

    def to_json(self) -> dict[str, Any]:
        """A minimal HF-style config.json that round-trips through from_json."""
        d: dict[str, Any] = dict(self.raw) if self.raw else {}
        if self.stack is not None:
            return d
        d.update({
            "hidden_size": self.hidden_size, "intermediate_size": self.intermediate_size,
            "num_hidden_layers": self.num_layers, "num_attention_heads": self.num_heads,
            "num_key_value_heads": self.num_kv_heads, "head_dim": self.head_dim, "vocab_size": self.vocab_size,
            "rms_norm_eps": self.rms_norm_eps, "rope_theta": self.rope_theta,
            "tie_word_embeddings": self.tie_word_embeddings,
        })
        if "model_type" not in d and "architectures" not in d:
            d["model_type"] = self.architecture.value
        if self.max_position_embeddings:
            d["max_position_embeddings"] = self.max_position_embeddings
        if self.quantization_bits:
            d["quantization"] = {"bits": self.quantization_bits}
            if self.quantization_group_size:
                d["quantization"]["group_size"] = self.quantization_group_size
        return d

    # ---- derived quantities ----------------------------------------------------------------
    @property
    def groups(self) -> int:
        if self.stack is not None:
            return max(lay.mixer.groups for lay in self.stack.layers)
        return self.num_heads // self.num_kv_heads

    @property
    def rotary_dim(self) -> int:
        return int(round(self.head_dim * self.partial_rotary_factor)) & ~1

    @property
    def attn_scale(self) -> float:
        if self.mla is not None:
            m = self.yarn.softmax_mscale() if self.yarn else 1.0
            return self.mla.q_head_dim ** -0.5 * m * m
        return float(self.query_pre_attn_scalar or self.head_dim) ** -0.5

    @property
    def is_moe(self) -> bool:
        return self.moe is not None

    @property
    def norm_weight_offset(self) -> float:
        return 1.0 if self.architecture is Architecture.GEMMA2 else 0.0

    @property
    def embed_scale(self) -> float:
        return math.sqrt(self.hidden_size) if self.architecture is Architecture.GEMMA2 else 1.0

    @property
    def mlp_activation(self) -> str:
        return "gelu_tanh" if self.architecture is Architecture.GEMMA2 else "silu"

    def mrope_section_resolved(self) -> tuple[int, int, int]:
        if self.mrope_section:
            return tuple(max(0, s) for s in self.mrope_section)  # type: ignore[return-value]
        half = self.rotary_dim // 2
        base, rem = divmod(half, 3)
        return (base + (rem > 0), base + (rem > 1), base)


def _plain_inv_freq(dim: int, theta: float) -> list[float]:
    return [1.0 / theta ** ((2 * i) / dim) for i in range(dim // 2)]


def rescale_frequencies(freqs: list[float], rs: RopeScaling) -> list[float]:
    """Llama-3 frequency bands: wavelengths above original / low are stretched by `factor`, those below original / high stay, and between
    the two the frequencies are mixed."""
    low_wl = rs.original_context / rs.low_freq_factor
    high_wl = rs.original_context / rs.high_freq_factor
    out = []
    for inv in freqs:
        wl = 2.0 * math.pi / inv
        if wl > low_wl:
            out.append(inv / rs.factor)
        elif wl < high_wl:
            out.append(inv)
        else:
            smooth = (rs.original_context / wl - rs.low_freq_factor) / (rs.high_freq_factor - rs.low_freq_factor)
            out.append((1.0 - smooth) * inv / rs.factor + smooth * inv)
    return out


def build_rope(cfg: ModelConfig) -> RopeSpec:
    """Inverse-frequency table for the configured RoPE variant (standard, partial / interleaved, Llama-3
    frequency-band scaling, YaRN). Parity: candle-llm/src/primitives/rope.rs:35-170, config.rs:540-575."""
    if cfg.mla is not None:
        dim = cfg.mla.qk_rope_head_dim
        if cfg.yarn is None:
            return RopeSpec(tuple(_plain_inv_freq(dim, cfg.rope_theta)), dim, True)
        y = cfg.yarn

        def correction_dim(rot: float) -> float:
            return dim * math.log(y.original_context / (rot * 2.0 * math.pi)) / (2.0 * math.log(cfg.rope_theta))

        low = max(0.0, math.floor(correction_dim(y.beta_fast)))
        high = min(float(dim - 1), math.ceil(correction_dim(y.beta_slow)))
        span = 1e-3 if abs(high - low) < 1e-3 else high - low
        out = []
        for i, extra in enumerate(_plain_inv_freq(dim, cfg.rope_theta)):
            ramp = min(1.0, max(0.0, (i - low) / span))
            out.append(extra / y.factor * ramp + extra * (1.0 - ramp))
        return RopeSpec(tuple(out), dim, True)
    rd = cfg.rotary_dim
    if rd < cfg.head_dim or cfg.architecture.rope_interleaved:
        return RopeSpec(tuple(_plain_inv_freq(rd, cfg.rope_theta)), rd, cfg.architecture.rope_interleaved)
    base = _plain_inv_freq(cfg.head_dim, cfg.rope_theta)
    rs = cfg.rope_scaling
    if rs is None:
        return RopeSpec(tuple(base), cfg.head_dim, False)
    out = rescale_frequencies(base, rs)
    return RopeSpec(tuple(out), cfg.head_dim, False)
