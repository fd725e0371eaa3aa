"""Model configuration: ``config.ini`` / ``config.json`` parsing and dtype-string handling.

The checkpoint directory contract is the reference's: one ``config.ini`` whose single
section name selects the model family, plus raw ``.bin`` tensors.  The keys and their
defaults follow ``src/models/common_decoder.h:167-270`` of the reference; the dtype
vocabulary follows ``include/dtype.h:18-36`` and
``src/xfastertransformer/automodel.py:19-47``.

Unlike the reference, where every (family, weight type, kv type) triple is a C++ template
instantiation, here all of this is *data*: one `ModelConfig` drives one generic decoder.

Designs that describe themselves layer by layer come as ``config.json`` (plus ``model.safetensors``) instead: its
``layers`` list becomes `ModelConfig.layers`, one `LayerConfig` per layer, and every size and constant is per layer.
"""
from __future__ import annotations

import configparser
import json
import math
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

# dtype strings accepted by AutoModel (reference automodel.py:20-37)
WEIGHT_DTYPES = (
    "fp16", "bf16", "int8", "w8a8", "int4", "nf4",
    "bf16_fp16", "bf16_int8", "bf16_w8a8", "bf16_int4", "bf16_nf4",
    "w8a8_int8", "w8a8_int4", "w8a8_nf4", "fp8_e4m3",
    "fp32",                           # everything in 32 bits: layered designs on a GPU, any family on CPU
)
KV_DTYPES = ("fp16", "bf16", "int8")

# config.ini section names registered by the reference (model_factory.h / models.cpp:1022)
MODEL_TYPES = (
    "llama", "yarn_llama", "gemma", "qwen", "qwen2", "qwen3", "qwen3_moe", "mixtral",
    "deepseek_moe", "baichuan", "chatglm", "chatglm2", "chatglm3", "chatglm4", "gpt",
    "telechat",
)

# config.json "architecture" -> model type
ARCHITECTURES = {"Kafipel": "kafipel", "Vepivik": "vepivik", "Botusun": "botusun", "Dagezen": "dagezen"}

# what a design fixes about its mixers and experts beside what its config.json says
MIXER_TRAITS = {"botusun": {"attention": dict(values_from_keys=True, qk_bias=True, qk_norm=True, sink=0.0)},
                "dagezen": {"latent_attention": dict(head_gate=True, sinks=True)}}
MOE_TRAITS = {"botusun": dict(act="silu", gated=True, scoring="sigmoid", renorm=False, correction=True),
              "dagezen": dict(act="gelu_erf", scoring="chosen", router_bias=True)}
DENSE_TRAITS = {"dagezen": dict(act="clamped", ff_bias=True)}


def split_hybrid_dtype(dtype: str) -> Tuple[str, str]:
    """``"bf16_int8"`` -> (prefill dtype, decode dtype); plain names map to themselves.

    ``fp8_e4m3`` contains an underscore but is a single type (reference
    ``hybrid_model.h:46-83`` registers only the pairs listed in `WEIGHT_DTYPES`).
    """
    if dtype not in WEIGHT_DTYPES:
        raise ValueError(f"AutoModel don't support {dtype}.")
    if dtype == "fp8_e4m3" or "_" not in dtype:
        return dtype, dtype
    a, b = dtype.split("_", 1)
    return a, b


def _to_bool(v) -> bool:
    if isinstance(v, bool):
        return v
    s = str(v).strip().lower()
    if s in ("1", "true", "yes", "on"):
        return True
    if s in ("0", "false", "no", "off", ""):
        return False
    return bool(float(s))


@dataclass
class RopeConfig:
    theta: float = 10000.0
    scaling_type: str = ""            # "", "linear", "yarn", "dynamic"
    scaling_factor: float = 1.0
    original_max_pos: int = 2048
    beta_fast: float = 32.0
    beta_slow: float = 1.0
    mscale: float = 1.0
    mscale_all_dim: float = 1.0


@dataclass(frozen=True)
class RotaryConfig:
    """Rotary positions of one layer: the first `dims` dimensions of each head (of the rotated part, in latent attention),
    base, optional scaling; `style` "half" pairs dimension i with i + dims/2, "interleaved" 2i with 2i + 1.
    `scaling` "yarn" uses `fast` and `slow`; "banded" keeps the frequencies of wavelengths below original / `high`, divides
    those above original / `low` by the factor, with a ramp between them (the scheme of Llama 3.1)."""
    dims: int
    base: float
    factor: float = 0.0               # 0: no scaling
    original: float = 0.0
    fast: float = 32.0
    slow: float = 1.0
    style: str = "half"
    scaling: str = "yarn"
    low: float = 1.0
    high: float = 4.0


@dataclass(frozen=True)
class MixerConfig:
    """Token mixer of one layer.  `window` 0: every earlier position is visible; otherwise position i sees j <= i when
    i - j < window or j < keep_first.  `softcap` 0: scores are not capped.  `kv_from` >= 0: this layer has queries only
    and reads the keys and values of that layer.

    `kind` "latent": keys and values come from one latent of `kv_rank` values per token, expanded per head to `dim` key and
    `vdim` value dimensions, plus `rot_dim` rotated key dimensions that all heads share (kv_heads is 1: one cache row per
    token).  `gate`: the concatenated heads are multiplied with sigmoid(W_g h); `head_gate`: each head with one such value.
    `sinks`: a learned sink per head joins the softmax.

    `conv` > 0: queries and keys go through a causal convolution of that many taps, channel by channel, straight after
    their projections (`qk_bias`: which have biases).  `values_from_keys`: the values are the keys as they leave it, before
    norm and rotation.  `qk_norm`: RMS norm per head in front of the rotation.  `sink`: score of a softmax sink that all
    heads share and that is no tensor.

    `kind` "gla": gated linear attention, heads of `dim` x `vdim` states that decay per key channel by
    sigmoid(z)^(1 / `tau`); no cache, one fp32 state per sequence.

    `kind` "time_mix": a recurrence of the same shape over mixes of each token's input with the previous one's, with decays
    exp(-exp(z)) and a bonus for the current token.

    `kind` "ssd": a state-space recurrence (Mamba-2), heads of `dim` x `vdim` states with one decay per head and token; keys
    and queries are shared by the heads of each of `groups`, inputs pass a convolution of `conv` taps, and outputs a norm in
    `norm_groups` parts.

    `kind` "talking": attention whose values are its keys, with norms over whole projections, a logarithmic distance bias and
    weights that are mixed between the heads.

    `kind` "parallel": the `parts`, side by side on the same input, their outputs summed with the factors `part_scales`."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    kind: str = "attention"
    softcap: float = 0.0
    window: int = 0
    keep_first: int = 0
    rot: Optional[RotaryConfig] = None
    kv_from: int = -1
    kv_rank: int = 0
    rot_dim: int = 0
    gate: bool = False
    head_gate: bool = False
    sinks: bool = False
    conv: int = 0
    values_from_keys: bool = False
    qk_bias: bool = False
    qk_norm: bool = False
    sink: Optional[float] = None
    tau: float = 1.0
    groups: int = 1
    norm_groups: int = 1
    parts: Tuple["MixerConfig", ...] = ()
    part_scales: Tuple[float, ...] = ()

    @property
    def has_kv(self) -> bool:
        """Whether a layer with this mixer keeps keys and values (its own or another layer's)."""
        return self.kind not in ("gla", "time_mix", "ssd") and (not self.parts or any(p.has_kv for p in self.parts))

    def kv_shape(self) -> tuple:
        """What two layers must agree on for one to read the other's cache."""
        if self.kind == "latent":
            return self.kind, self.kv_rank, self.rot_dim, self.rot
        return self.kind, self.kv_heads, self.dim, self.vdim


@dataclass(frozen=True)
class MoeConfig:
    """Mixture of experts of one layer: scores from `experts` router logits (`scoring`: softmax over them, or the sigmoid of
    each; "chosen": softmax over the chosen ones' logits alone), the `top` best, weighted with their scores (`renorm`: divided by their sum) times `scale`, and (`shared` > 0)
    one more expert that every token uses.  `correction`: a tensor added to the scores for the choice alone.  `groups` > 1:
    only experts of the `keep_groups` groups with the best sum of two choice scores can be chosen.  An expert is
    down(act(up x)), or with `gated` down(act(gate x) * up x)."""
    experts: int
    top: int
    ff: int
    shared: int = 0
    act: str = "relu2"
    gated: bool = False
    scoring: str = "softmax"
    renorm: bool = True
    scale: float = 1.0
    correction: bool = False
    groups: int = 1
    keep_groups: int = 1
    router_bias: bool = False


@dataclass(frozen=True)
class LayerConfig:
    mixer: MixerConfig
    ff: int = 0                       # width of a dense feed-forward; 0: none
    ff_kind: str = "dense"
    moe: Optional[MoeConfig] = None
    act: str = "silu"                 # of the dense feed-forward's gate; "clamped" takes `limit` (see ops.linear_gated)
    limit: float = 0.0
    ff_bias: bool = False


@dataclass(frozen=True)
class LoopConfig:
    """Layers start .. stop - 1 run `times` times in a row; every pass has a cache and states of its own."""
    start: int
    stop: int
    times: int


@dataclass
class ModelConfig:
    model_type: str = "llama"
    head_num: int = 0
    kv_head_num: int = 0
    size_per_head: int = 0
    hidden_size: int = 0
    inter_size: int = 0
    num_layer: int = 0
    vocab_size: int = 0
    max_pos_seq_len: int = 0
    model_max_length: int = 0
    seq_length: int = -1              # Qwen-1 training length for log-n / NTK
    use_logn_attn: bool = True
    use_dynamic_ntk: bool = True
    layernorm_eps: float = 1e-6
    activation_type: str = "silu"
    start_id: int = 0
    end_id: int = 0
    pad_id: int = -1
    weight_data_type: str = "fp16"    # storage type of the .bin files
    quant_qweight_data_type: str = ""
    quant_scales_data_type: str = ""
    quant_zeros_data_type: str = ""
    quant_groupsize: int = -1
    rope: RopeConfig = field(default_factory=RopeConfig)
    # MoE
    sparse_experts: int = 8
    dense_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = False
    first_k_dense_replace: int = 0
    topk_group: int = 0
    n_group: int = 0
    topk_method: str = ""
    scoring_func: str = ""
    routed_scaling_factor: float = 1.0
    # MLA
    q_lora_rank: int = 0
    kv_lora_rank: int = 0
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    # Qwen3
    do_qk_norm: bool = False
    # layered designs (config.json): one entry per layer; the scalar sizes above then hold the first layer's
    layers: List[LayerConfig] = field(default_factory=list)
    embed_scale: float = 1.0
    residual_mult: float = 1.0        # factor of every sublayer's output in the residual sum
    residual_carry: float = 1.0       # factor of the stream itself in the residual sum
    logit_softcap: float = 0.0        # > 0: logits become cap * tanh(logits / cap)
    loop: Optional[LoopConfig] = None
    side_dim: int = 0                 # > 0: each layer also gets so many values of the token's own side embedding
    # raw key/value pairs (for family-specific look-ups, like DecoderContext::GetAttr)
    raw: Dict[str, str] = field(default_factory=dict)

    # ---- derived ----------------------------------------------------------------------
    @property
    def is_mla(self) -> bool:
        return self.qk_nope_head_dim > 0 and self.qk_rope_head_dim > 0

    def runs(self) -> List[Tuple[int, int]]:
        """(layer, pass) in the order they run; pass -1: outside the loop."""
        n, loop = len(self.layers) or self.num_layer, self.loop
        if loop is None:
            return [(i, -1) for i in range(n)]
        return [(i, -1) for i in range(loop.start)] + \
            [(i, t) for t in range(loop.times) for i in range(loop.start, loop.stop)] + [(i, -1) for i in range(loop.stop, n)]

    @property
    def q_size(self) -> int:
        return self.head_num * self.size_per_head

    @property
    def kv_size(self) -> int:
        return self.kv_head_num * self.size_per_head

    @property
    def attn_scale(self) -> float:
        """Softmax scale.  MLA: 1/sqrt(nope+rope) * mscale^2 where the reference hard-wires
        the YaRN factor 40 (``common_decoder.h:272-274``); here the factor comes from the
        config so other factors work too (identical for DeepSeek-V3/R1, factor 40)."""
        if self.is_mla:
            base = 1.0 / math.sqrt(self.qk_nope_head_dim + self.qk_rope_head_dim)
            if self.rope.scaling_type == "yarn" and self.rope.scaling_factor > 1:
                m = 0.1 * self.rope.mscale_all_dim * math.log(self.rope.scaling_factor) + 1.0
                return base * m * m
            return base
        return 1.0 / math.sqrt(self.size_per_head)

    def get(self, key: str, default=None):
        return self.raw.get(key, default)

    # ---- io ---------------------------------------------------------------------------
    @classmethod
    def load(cls, path: str) -> "ModelConfig":
        """The configuration of a model directory: ``config.json`` of a layered design, else ``config.ini``."""
        js = os.path.join(path, "config.json")
        if os.path.isfile(js) and not os.path.exists(os.path.join(path, "config.ini")):
            return cls.from_json(path)
        return cls.from_ini(path)

    @classmethod
    def from_json(cls, path: str) -> "ModelConfig":
        with open(path if path.endswith(".json") else os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f), path)

    @classmethod
    def from_dict(cls, d: dict, where: str = "config.json") -> "ModelConfig":
        """A layered design from the contents of its ``config.json``."""
        arch = d.get("architecture")
        if arch not in ARCHITECTURES:
            raise ValueError(f"unsupported architecture {arch!r} in {where}; known: {sorted(ARCHITECTURES)}")
        layers = [_layer_config(i, e, ARCHITECTURES[arch]) for i, e in enumerate(d["layers"])]
        loop = None
        if d.get("loop"):
            loop = LoopConfig(*(int(d["loop"][k]) for k in ("start", "stop", "times")))
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                raise ValueError(f"loop {d['loop']} does not fit {len(layers)} layers")
            if any(l.mixer.kv_from >= 0 for l in layers):
                raise ValueError("layers that read another layer's keys do not combine with a loop")
        for i, l in enumerate(layers):
            j = l.mixer.kv_from
            if j >= 0:
                src = layers[j].mixer if j < i else None
                if src is None or src.kv_from >= 0:
                    raise ValueError(f"layer {i}: kv_from {j} is not an earlier layer with keys and values of its own")
                if src.kv_shape() != l.mixer.kv_shape():
                    raise ValueError(f"layer {i}: heads differ from those of layer {j}, whose keys it reads")
        m = layers[0].mixer
        return cls(model_type=ARCHITECTURES[arch], head_num=m.heads, kv_head_num=m.kv_heads, size_per_head=m.dim,
                   v_head_dim=m.vdim, hidden_size=int(d["width"]), inter_size=layers[0].ff, num_layer=len(layers),
                   vocab_size=int(d["vocab"]), layernorm_eps=float(d["norm"]["eps"]), start_id=-1, end_id=-1,
                   weight_data_type="bf16", layers=layers, raw=d,
                   embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                   residual_mult=float(d.get("residual_mult", 1.0)), residual_carry=float(d.get("postln_alpha", 1.0)),
                   logit_softcap=float(d.get("logit_softcap") or 0.0), loop=loop,
                   side_dim=int((d.get("token_side") or {}).get("dim", 0)))

    @classmethod
    def from_ini(cls, path: str) -> "ModelConfig":
        ini = path if path.endswith(".ini") else os.path.join(path, "config.ini")
        if not os.path.exists(ini):
            raise FileNotFoundError(f"config.ini not found under {path}")
        cp = configparser.ConfigParser()
        cp.read(ini)
        secs = cp.sections()
        if not secs:
            raise ValueError(f"{ini} has no section")
        sec = secs[0]
        if sec not in MODEL_TYPES:
            raise ValueError(f"unsupported model type [{sec}] in {ini}")
        kv = {k: v for k, v in cp[sec].items()}

        def gi(k, d=0):
            return int(float(kv[k])) if k in kv and kv[k] != "" else d

        def gf(k, d=0.0):
            return float(kv[k]) if k in kv and kv[k] != "" else d

        def gs(k, d=""):
            return kv.get(k, d)

        def gb(k, d=False):
            return _to_bool(kv[k]) if k in kv else d

        head_num = gi("head_num")
        size_per_head = gi("size_per_head")
        max_pos = gi("max_pos_seq_len", 0)
        # The reference reads only `layernorm_eps` (default 1e-6) and ignores the
        # `rms_norm_eps` some converters write; honour both, in that order.
        eps = gf("layernorm_eps", gf("rms_norm_eps", 1e-6))
        c = cls(
            model_type=sec,
            head_num=head_num,
            kv_head_num=gi("kv_head_num", head_num),
            size_per_head=size_per_head,
            hidden_size=gi("hidden_size", head_num * size_per_head),
            inter_size=gi("inter_size"),
            num_layer=gi("num_layer"),
            vocab_size=gi("vocab_size"),
            max_pos_seq_len=max_pos,
            model_max_length=gi("model_max_length", max_pos),
            seq_length=gi("seq_length", -1),
            use_logn_attn=gb("use_logn_attn", True),
            use_dynamic_ntk=gb("use_dynamic_ntk", True),
            layernorm_eps=eps,
            activation_type=gs("activation_type", "silu").lower(),
            start_id=gi("start_id", 0),
            end_id=gi("end_id", gi("start_id", 0)),
            pad_id=gi("pad_id", -1),
            weight_data_type=gs("weight_data_type", "fp16").lower(),
            quant_qweight_data_type=gs("quant_qweight_data_type", ""),
            quant_scales_data_type=gs("quant_scales_data_type", ""),
            quant_zeros_data_type=gs("quant_zeros_data_type", ""),
            quant_groupsize=gi("quant_groupsize", -1),
            rope=RopeConfig(
                theta=gf("rope_theta", 10000.0),
                scaling_type=gs("rope_scaling_type", gs("rope_type", "")).lower(),
                scaling_factor=gf("rope_scaling_factor", gf("scaling_factor", 1.0)),
                original_max_pos=gi("rope_scaling_original_max_position_embeddings", 2048),
                beta_fast=gf("rope_scaling_beta_fast", 32),
                beta_slow=gf("rope_scaling_beta_slow", 1),
                mscale=gf("rope_scaling_mscale", 1.0),
                mscale_all_dim=gf("rope_scaling_mscale_all_dim", 1.0),
            ),
            sparse_experts=gi("sparse_experts", 8),
            dense_experts=gi("dense_experts", 0),
            num_experts_per_tok=gi("num_experts_per_tok", 0),
            moe_intermediate_size=gi("moe_intermediate_size", 0),
            norm_topk_prob=gb("norm_topk_prob", False),
            first_k_dense_replace=gi("first_k_dense_replace", 0),
            topk_group=gi("topk_group", 0),
            n_group=gi("n_group", 0),
            topk_method=gs("topk_method", ""),
            scoring_func=gs("scoring_func", ""),
            routed_scaling_factor=gf("routed_scaling_factor", 1.0),
            q_lora_rank=gi("q_lora_rank", 0),
            kv_lora_rank=gi("kv_lora_rank", 0),
            qk_nope_head_dim=gi("qk_nope_head_dim", 0),
            qk_rope_head_dim=gi("qk_rope_head_dim", 0),
            v_head_dim=gi("v_head_dim", 0),
            do_qk_norm=gb("do_qk_norm", False),
            raw=kv,
        )
        if c.quant_qweight_data_type in ("int8", "uint4"):
            if c.quant_scales_data_type != "fp32" or c.quant_zeros_data_type != "fp32":
                raise ValueError("quantised checkpoints need fp32 scales and zeros")
            if c.quant_groupsize != -1:
                raise ValueError("Quantization with groupsize is not supported.")
        if c.model_type == "mixtral" and c.num_experts_per_tok == 0:
            c.num_experts_per_tok = 2
        if c.is_mla and c.v_head_dim == 0:
            c.v_head_dim = c.size_per_head
        return c

    def to_ini(self, path: str, extra: Optional[Dict[str, str]] = None) -> None:
        """Write a config.ini the way the converters do (one section = model type); config.json for a layered design."""
        if self.layers:
            os.makedirs(path, exist_ok=True)
            with open(os.path.join(path, "config.json"), "w") as f:
                json.dump(self.raw, f, indent=1)
            return
        cp = configparser.ConfigParser()
        d: Dict[str, str] = dict(self.raw)
        d.update({
            "head_num": str(self.head_num),
            "kv_head_num": str(self.kv_head_num),
            "size_per_head": str(self.size_per_head),
            "hidden_size": str(self.hidden_size),
            "inter_size": str(self.inter_size),
            "num_layer": str(self.num_layer),
            "vocab_size": str(self.vocab_size),
            "max_pos_seq_len": str(self.max_pos_seq_len),
            "layernorm_eps": repr(self.layernorm_eps),
            "activation_type": self.activation_type,
            "start_id": str(self.start_id),
            "end_id": str(self.end_id),
            "weight_data_type": self.weight_data_type,
            "rope_theta": repr(self.rope.theta),
        })
        if self.rope.scaling_type:
            d.update({
                "rope_scaling_type": self.rope.scaling_type,
                "rope_scaling_factor": repr(self.rope.scaling_factor),
                "rope_scaling_original_max_position_embeddings": str(self.rope.original_max_pos),
                "rope_scaling_beta_fast": repr(self.rope.beta_fast),
                "rope_scaling_beta_slow": repr(self.rope.beta_slow),
                "rope_scaling_mscale": repr(self.rope.mscale),
                "rope_scaling_mscale_all_dim": repr(self.rope.mscale_all_dim),
            })
        if self.model_type in ("mixtral", "qwen3_moe", "deepseek_moe"):
            d.update({
                "sparse_experts": str(self.sparse_experts),
                "dense_experts": str(self.dense_experts),
                "num_experts_per_tok": str(self.num_experts_per_tok),
                "moe_intermediate_size": str(self.moe_intermediate_size),
                "norm_topk_prob": str(self.norm_topk_prob),
            })
        if self.is_mla:
            d.update({
                "q_lora_rank": str(self.q_lora_rank),
                "kv_lora_rank": str(self.kv_lora_rank),
                "qk_nope_head_dim": str(self.qk_nope_head_dim),
                "qk_rope_head_dim": str(self.qk_rope_head_dim),
                "v_head_dim": str(self.v_head_dim),
                "first_k_dense_replace": str(self.first_k_dense_replace),
                "topk_group": str(self.topk_group),
                "n_group": str(self.n_group),
                "topk_method": self.topk_method,
                "scoring_func": self.scoring_func,
                "routed_scaling_factor": repr(self.routed_scaling_factor),
            })
        if self.do_qk_norm:
            d["do_qk_norm"] = "1"
        if self.model_type == "qwen":
            d.update({"seq_length": str(self.seq_length), "use_logn_attn": str(int(self.use_logn_attn)),
                      "use_dynamic_ntk": str(int(self.use_dynamic_ntk))})
        if extra:
            d.update(extra)
        cp[self.model_type] = d
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.ini"), "w") as f:
            cp.write(f)


def _rotary(i: int, m: dict, width: int, style: str) -> Optional[RotaryConfig]:
    if not m.get("rot"):
        return None
    r, sc = m["rot"], m["rot"].get("scaling") or {}
    rot = RotaryConfig(int(r["dims"]), float(r["base"]), float(sc.get("factor", 0.0)), float(sc.get("original", 0.0)),
                       float(sc.get("fast", 32.0)), float(sc.get("slow", 1.0)), style, "banded" if "low" in sc else "yarn",
                       float(sc.get("low", 1.0)), float(sc.get("high", 4.0)))
    if rot.dims % 2 or rot.dims > width:
        raise ValueError(f"layer {i}: rotary dims {rot.dims} do not fit heads of {width}")
    return rot


def _mixer_config(i: int, kind: str, m: dict, model_type: str) -> MixerConfig:
    if kind == "parallel":
        parts = tuple(_mixer_config(i, k, m[name], model_type) for name, k in PARALLEL_PARTS)
        q = parts[0]
        return MixerConfig(kind="parallel", heads=q.heads, kv_heads=q.kv_heads, dim=q.dim, vdim=q.vdim, scale=q.scale, window=q.window,
                           parts=parts, part_scales=tuple(float(m.get(name + "_scale", 1.0)) for name, _ in PARALLEL_PARTS))
    if kind not in ("attention", "latent_attention", "gla", "time_mix", "mamba2", "talking"):
        raise ValueError(f"layer {i}: unsupported mixer type {kind!r}")
    mask = m.get("mask") or {}
    dim = int(m["state"] if kind == "mamba2" else m["dim"])
    scale = {"gla": dim ** -0.5, "mamba2": 1.0, "time_mix": 1.0}.get(kind)
    common = dict(heads=int(m["heads"]), dim=dim, vdim=int(m.get("vdim", dim)),
                  scale=float(m["scale"]) if scale is None else scale,
                  window=int(mask.get("size") or 0), keep_first=int(mask.get("keep_first") or 0),
                  softcap=float(m.get("softcap") or 0.0), kv_from=-1 if m.get("kv_from") is None else int(m["kv_from"]),
                  conv=int(m.get("conv") or 0), **MIXER_TRAITS.get(model_type, {}).get(kind, {}))
    if kind == "attention":
        return MixerConfig(kv_heads=int(m.get("kv_heads", m["heads"])), rot=_rotary(i, m, dim, "half"), **common)
    if kind == "latent_attention":
        rd = int(m["rot_dim"])
        mixer = MixerConfig(kind="latent", kv_heads=1, rot=_rotary(i, m, rd, "interleaved"), kv_rank=int(m["kv_rank"]), rot_dim=rd,
                            **{"gate": True, **common})
        if mixer.keep_first or mixer.softcap:
            raise ValueError(f"layer {i}: latent attention has no kept first keys and no cap on the scores")
        return mixer
    if kind == "gla":
        return MixerConfig(kind="gla", kv_heads=common["heads"], tau=float(m["tau"]), **common)
    if kind == "time_mix":
        return MixerConfig(kind="time_mix", kv_heads=common["heads"], **common)
    if kind == "mamba2":
        mixer = MixerConfig(kind="ssd", kv_heads=common["heads"], groups=int(m["groups"]), norm_groups=int(m["norm_groups"]), **common)
        if mixer.groups < 1 or mixer.heads % mixer.groups or mixer.norm_groups < 1 or mixer.heads * mixer.vdim % mixer.norm_groups:
            raise ValueError(f"layer {i}: {mixer.heads} heads of {mixer.vdim} in {mixer.groups} groups, normalised in {mixer.norm_groups}")
        return mixer
    return MixerConfig(kind="talking", kv_heads=int(m.get("kv_heads", m["heads"])), values_from_keys=True, **common)


# what a parallel mixer consists of: (key in its entry and prefix of its tensors, mixer type)
PARALLEL_PARTS = (("left", "talking"), ("right", "time_mix"))


def _check_mixer(i: int, mixer: MixerConfig) -> None:
    if mixer.heads % mixer.kv_heads:
        raise ValueError(f"layer {i}: {mixer.heads} query heads over {mixer.kv_heads} key/value heads")
    if mixer.values_from_keys and (mixer.dim != mixer.vdim or mixer.kv_from >= 0):
        raise ValueError(f"layer {i}: values that are keys have the keys' size and a cache of their own")
    if mixer.conv and not mixer.values_from_keys and mixer.kind != "ssd":
        raise ValueError(f"layer {i}: a short convolution is for layers whose values are their keys and for state-space layers")
    if mixer.kind == "talking" and (mixer.keep_first or mixer.softcap or mixer.conv):
        raise ValueError(f"layer {i}: mixed heads have no kept first keys, no cap and no convolution")
    if mixer.kind == "time_mix" and mixer.dim != mixer.vdim:
        raise ValueError(f"layer {i}: time mixing has values of the keys' size")
    for p in mixer.parts:
        _check_mixer(i, p)


def _layer_config(i: int, e: dict, model_type: str) -> LayerConfig:
    """One entry of config.json's ``layers``."""
    mixer = _mixer_config(i, e.get("type"), e["mixer"], model_type)
    _check_mixer(i, mixer)
    f = e.get("mlp")
    if not f:
        return LayerConfig(mixer)
    if f.get("kind") == "dense":
        return LayerConfig(mixer, int(f["ff"]), "dense", limit=float(f.get("limit") or 0.0), **DENSE_TRAITS.get(model_type, {}))
    if f.get("kind") != "moe":
        raise ValueError(f"layer {i}: unsupported feed-forward {f.get('kind')!r}")
    r = f["router"]
    groups = r.get("groups") or {}
    moe = MoeConfig(experts=int(r["experts"]), top=int(r["top"]), ff=int(f["expert"]["ff"]),
                    shared=int((f.get("shared") or {}).get("ff", 0)), scale=float(r.get("scale", 1.0)),
                    groups=int(groups.get("count", 1)), keep_groups=int(groups.get("keep", 1)), **MOE_TRAITS.get(model_type, {}))
    if moe.groups < 1 or moe.experts % moe.groups or not 0 < moe.keep_groups <= moe.groups:
        raise ValueError(f"layer {i}: {moe.keep_groups} of {moe.groups} groups of {moe.experts} experts")
    if not 0 < moe.top <= moe.experts // moe.groups * moe.keep_groups:
        raise ValueError(f"layer {i}: {moe.top} of {moe.experts // moe.groups * moe.keep_groups} experts")
    return LayerConfig(mixer, 0, "moe", moe)
