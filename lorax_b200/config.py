"""Typed configuration objects.

Two dataclasses replace the import-time environment globals of the reference
(`server/lorax_server/utils/state.py:12-38`, `utils/dist.py:8-14`,
`utils/graph.py:29-31`):

* :class:`ModelConfig` is the parsed HuggingFace ``config.json`` of the base model.
* :class:`EngineConfig` is every serving knob (launcher flags + environment),
  resolved once and passed explicitly.  Public flag names follow the reference
  launcher (`launcher/src/main.rs:273-655`).
"""

from __future__ import annotations

import dataclasses
import json
import os
from dataclasses import dataclass, field
from typing import Any, Callable, Dict, List, Optional, Tuple

# Architectures handled by the single config-driven decoder (models/decoder.py).
DECODER_MODEL_TYPES = (
    "llama", "mistral", "mixtral", "qwen2", "qwen", "gemma", "gemma2", "phi3", "phi",
    "cohere", "solar", "granite", "gpt2", "gpt_neox", "falcon", "RefinedWeb",
    "RefinedWebModel", "gpt_bigcode", "dbrx",
)


# Designs whose config.json lists its layers one by one, each with a mixer of its own (models/mixers.py).
MIXER_MODEL_TYPES = ("vabunex", "sapudra", "saredra", "fegolorn")


@dataclass
class MoeSpec:
    """Routed feed-forward: `experts` of width `ff`, `top` of them per token, chosen within the best `keep` of `groups` groups of
    neighbours (0: no groups), a group counting by the sum of its `group_top` largest scores.  `score`: "sigmoid" (plus a correction
    that takes part in the choice only) or "softmax" over all experts.  The weights are the chosen scores, normalised if `renorm`, times
    `scale`.  `gated`: an expert is down(act(gate) * up) instead of down(act(up)).  `shared_ff`: width of the expert that every token
    takes beside them (0: none), with a weight of its own (`shared_gate`) or with weight one.  `bias`: the router's logits have one."""
    experts: int
    top: int
    ff: int
    scale: float = 1.0
    groups: int = 0
    keep: int = 0
    shared_ff: int = 0
    score: str = "sigmoid"
    renorm: bool = True
    group_top: int = 2
    gated: bool = False
    bias: bool = False
    shared_gate: bool = True

    def __post_init__(self):
        if not 1 <= self.top <= self.experts:
            raise ValueError(f"{self.top} of {self.experts} experts")
        if self.groups:
            if self.experts % self.groups or not 1 <= self.keep <= self.groups:
                raise ValueError(f"{self.experts} experts in {self.groups} groups of which {self.keep} are kept")
            if self.keep * (self.experts // self.groups) < self.top:
                raise ValueError(f"{self.keep} groups of {self.experts // self.groups} experts cannot give {self.top}")


@dataclass
class LayerSpec:
    """One layer of a design whose layers differ: the kind of mixer, the mixer's sizes and constants, and its feed-forward: dense of
    width `ff` (0: none; `gated`: act(gate) * up), or routed experts (`moe`).  `act`: activation of the dense one (empty: the model's), with
    its `limit` where it has one.  `weights_of`: the layer whose tensors it uses (its cache or state is its own)."""
    mixer: str
    params: Dict[str, Any]
    ff: int = 0
    moe: Optional[MoeSpec] = None
    gated: bool = False
    act: str = ""
    limit: float = 0.0
    weights_of: Optional[int] = None


@dataclass
class ModelConfig:
    model_type: str = "llama"
    vocab_size: int = 32000
    hidden_size: int = 4096
    intermediate_size: int = 11008
    num_hidden_layers: int = 32
    num_attention_heads: int = 32
    num_key_value_heads: Optional[int] = None
    head_dim: Optional[int] = None
    rms_norm_eps: float = 1e-5
    rope_theta: float = 10000.0
    rope_scaling: Optional[Dict[str, Any]] = None
    max_position_embeddings: int = 4096
    sliding_window: Optional[int] = None
    tie_word_embeddings: bool = False
    hidden_act: str = "silu"
    attention_bias: bool = False
    mlp_bias: bool = False
    # MoE (mixtral / dbrx)
    num_local_experts: int = 0
    num_experts_per_tok: int = 0
    # gemma-family quirks
    norm_weight_offset: float = 0.0          # gemma stores (w - 1)
    embedding_multiplier: float = 1.0        # gemma scales embeddings by sqrt(hidden)
    attn_logit_softcapping: Optional[float] = None
    final_logit_softcapping: Optional[float] = None
    query_pre_attn_scalar: Optional[float] = None
    # granite / cohere multipliers
    residual_multiplier: float = 1.0
    attention_multiplier: Optional[float] = None
    logits_scaling: float = 1.0
    logit_scale: float = 1.0
    # layer norm style: "rms" or "layernorm" (gpt2/neox/falcon/phi)
    norm_type: str = "rms"
    # rotary fraction (phi / neox partial rotary)
    partial_rotary_factor: float = 1.0
    # parallel attention+mlp blocks (falcon, neox, phi, cohere)
    parallel_residual: bool = False
    # learned absolute positions (gpt2, bigcode, opt); OPT's table starts at position_offset = 2
    learned_positions: bool = False
    position_offset: int = 0
    # ALiBi instead of any position embedding (bloom, mpt): bias -slope_h * distance on the attention scores
    alibi: bool = False
    alibi_bias_max: float = 8.0
    # LayerNorm right after the embedding lookup (bloom)
    embed_norm: bool = False
    # clamp of the fused QKV projection's output (mpt, dbrx)
    clip_qkv: Optional[float] = None
    # layer-by-layer designs: the layers, and (start, stop, times): layers start .. stop-1 run `times` times in a row
    layer_specs: Optional[List[LayerSpec]] = None
    layer_loop: Optional[Tuple[int, int, int]] = None
    # their residual: "parallel" (mixer and feed-forward read one norm of the stream, both are added to it), "pre" (the mixer, then the
    # feed-forward, each reading a norm of its own), "post" (each sublayer reads the stream itself, and a norm of its output, times
    # residual_multiplier, is added) or "sandwich" (each reads a norm of its own, and a second norm of its output is added)
    layer_style: str = "parallel"
    # "sandwich": each sublayer's output is multiplied by the sigmoid of a projection of its input before its norm, and by a vector after it
    residual_gate: bool = False
    layer_scale: bool = False
    norm_scalar: bool = False                # the norms of the stream have one number for all coordinates
    # vectors looked up by (previous token * mul_prev + token * mul_cur) mod buckets, added to the token's: (buckets, mul_prev, mul_cur)
    bigram: Optional[Tuple[int, int, int]] = None
    eos_token_id: Any = None
    bos_token_id: Any = None
    pad_token_id: Any = None
    torch_dtype: str = "bfloat16"
    quantization_config: Optional[Dict[str, Any]] = None
    extra: Dict[str, Any] = field(default_factory=dict)

    def __post_init__(self):
        if self.num_key_value_heads is None:
            self.num_key_value_heads = self.num_attention_heads
        if self.head_dim is None:
            self.head_dim = self.hidden_size // self.num_attention_heads

    # ------------------------------------------------------------------ sizes
    @property
    def q_size(self) -> int:
        return self.num_attention_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_key_value_heads * self.head_dim

    @property
    def rotary_dim(self) -> int:
        return int(self.head_dim * self.partial_rotary_factor)

    @property
    def layer_schedule(self) -> List[int]:
        """Layer indices in the order they run (a looped range counts every pass)."""
        n = self.num_hidden_layers
        if self.layer_loop is None:
            return list(range(n))
        a, b, k = self.layer_loop
        return list(range(a)) + list(range(a, b)) * k + list(range(b, n))

    @property
    def is_moe(self) -> bool:
        return self.num_local_experts > 0

    @property
    def attn_scale(self) -> float:
        if self.attention_multiplier is not None:
            return float(self.attention_multiplier)
        if self.query_pre_attn_scalar is not None:
            return float(self.query_pre_attn_scalar) ** -0.5
        return float(self.head_dim) ** -0.5

    # ------------------------------------------------------------------ io
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ModelConfig":
        d = dict(d)
        mt = d.get("model_type") or str(d.get("architecture", "")).lower() or "llama"
        if mt in MIXER_MODEL_TYPES:
            return cls(**_mixer_model_kwargs(mt, d))
        known = {f.name for f in dataclasses.fields(cls)}
        kw: Dict[str, Any] = {k: v for k, v in d.items() if k in known}
        extra = {k: v for k, v in d.items() if k not in known}
        # key aliases used by the older architectures
        alias = {
            "n_embd": "hidden_size", "n_layer": "num_hidden_layers", "n_head": "num_attention_heads",
            "n_positions": "max_position_embeddings", "n_inner": "intermediate_size",
            "layer_norm_epsilon": "rms_norm_eps", "layer_norm_eps": "rms_norm_eps",
            "num_kv_heads": "num_key_value_heads", "n_head_kv": "num_key_value_heads",
            "rotary_emb_base": "rope_theta", "rotary_pct": "partial_rotary_factor",
        }
        for src, dst in alias.items():
            if src in d and d[src] is not None and dst not in kw:
                kw[dst] = d[src]
        if kw.get("intermediate_size") is None:
            kw["intermediate_size"] = 4 * kw.get("hidden_size", 4096)
        if mt in ("gemma", "gemma2"):
            kw.setdefault("norm_weight_offset", 1.0)
            kw.setdefault("embedding_multiplier", float(kw.get("hidden_size", 4096)) ** 0.5)
            kw.setdefault("hidden_act", d.get("hidden_activation") or d.get("hidden_act", "gelu_pytorch_tanh"))
            kw.setdefault("tie_word_embeddings", True)
        if mt in ("gpt2", "gpt_bigcode"):
            kw.update(norm_type="layernorm", learned_positions=True, hidden_act=d.get("activation_function", "gelu_new"),
                      attention_bias=True, mlp_bias=True, tie_word_embeddings=True)
            if mt == "gpt_bigcode" and d.get("multi_query", True):
                kw["num_key_value_heads"] = 1
        if mt in ("gpt_neox",):
            kw.update(norm_type="layernorm", parallel_residual=d.get("use_parallel_residual", True),
                      attention_bias=True, mlp_bias=True, hidden_act=d.get("hidden_act", "gelu"))
        if mt in ("falcon", "RefinedWeb", "RefinedWebModel"):
            kw.update(norm_type="layernorm", parallel_residual=d.get("parallel_attn", True),
                      hidden_act="gelu", attention_bias=d.get("bias", False), mlp_bias=d.get("bias", False))
            # key/value heads: the 40b layout (new_decoder_architecture; "RefinedWeb" checkpoints imply it) names them, the
            # 7b layout has one shared head when multi_query is set, falcon-rw has as many as query heads
            new_arch = bool(d.get("new_decoder_architecture", mt == "RefinedWeb"))
            nh = kw.get("num_attention_heads", 32)
            if new_arch:
                kw["num_key_value_heads"] = d.get("num_kv_heads") or d.get("n_head_kv") or nh
            else:
                kw["num_key_value_heads"] = 1 if d.get("multi_query", True) else nh
            if d.get("alibi", False):
                raise NotImplementedError("falcon with ALiBi (falcon-rw): its bias is scaled with the scores, unlike bloom's")
            kw["rms_norm_eps"] = d.get("layer_norm_epsilon", 1e-5)
        if mt == "phi":
            kw.update(norm_type="layernorm", parallel_residual=True, attention_bias=True, mlp_bias=True,
                      hidden_act=d.get("hidden_act", "gelu_new"))
        if mt == "cohere":
            kw.update(norm_type="layernorm_nobias", parallel_residual=True, tie_word_embeddings=True)
        if mt == "qwen2":
            kw.setdefault("attention_bias", True)
        if mt == "granite":
            kw.setdefault("embedding_multiplier", d.get("embedding_multiplier", 1.0))
        if mt == "bloom":
            kw.update(norm_type="layernorm", alibi=True, embed_norm=True, attention_bias=True, mlp_bias=True, hidden_act="gelu_tanh",
                      tie_word_embeddings=True, hidden_size=d.get("hidden_size", d.get("n_embed", 4096)))
            kw["intermediate_size"] = 4 * kw["hidden_size"]
            kw.setdefault("max_position_embeddings", d.get("seq_length", 2048))
        if mt == "mpt":
            attn = d.get("attn_config", {}) or {}
            no_bias = d.get("no_bias", True)
            kw.update(hidden_size=d["d_model"], num_hidden_layers=d["n_layers"], num_attention_heads=d["n_heads"],
                      intermediate_size=int(d.get("expansion_ratio", 4) * d["d_model"]), max_position_embeddings=d.get("max_seq_len", 2048),
                      norm_type="layernorm_nobias" if no_bias else "layernorm", attention_bias=not no_bias, mlp_bias=not no_bias,
                      hidden_act="gelu", alibi=bool(attn.get("alibi", True)), alibi_bias_max=float(attn.get("alibi_bias_max", 8)),
                      clip_qkv=attn.get("clip_qkv"), learned_positions=not attn.get("alibi", True), tie_word_embeddings=True,
                      rms_norm_eps=d.get("layer_norm_epsilon", 1e-5))
            if attn.get("qk_ln"):
                raise NotImplementedError("mpt with qk_ln")
            ls = d.get("logit_scale")
            kw["logit_scale"] = 1.0 if ls is None else (float(d["d_model"]) ** -0.5 if ls == "inv_sqrt_d_model" else float(ls))
        if mt == "opt":
            if d.get("word_embed_proj_dim", d["hidden_size"]) != d["hidden_size"] or not d.get("do_layer_norm_before", True):
                raise NotImplementedError("opt with a projected embedding or post-layer-norm blocks (opt-350m)")
            kw.update(norm_type="layernorm", learned_positions=True, position_offset=2, attention_bias=d.get("enable_bias", True),
                      mlp_bias=d.get("enable_bias", True), hidden_act=d.get("activation_function", "relu"), intermediate_size=d["ffn_dim"],
                      tie_word_embeddings=d.get("tie_word_embeddings", True))
        if mt == "qwen":
            # first-generation Qwen: intermediate_size counts both halves of the gated MLP; fused c_attn with bias
            kw.update(intermediate_size=d["intermediate_size"] // 2, attention_bias=True, head_dim=d.get("kv_channels"),
                      max_position_embeddings=d.get("seq_length", d.get("max_position_embeddings", 8192)),
                      tie_word_embeddings=d.get("tie_word_embeddings", False))
        if mt == "dbrx":
            ffn = d.get("ffn_config", {})
            attn = d.get("attn_config", {})
            kw.update(hidden_size=d["d_model"], num_hidden_layers=d["n_layers"], num_attention_heads=d["n_heads"],
                      num_key_value_heads=attn.get("kv_n_heads", d["n_heads"]),
                      intermediate_size=ffn.get("ffn_hidden_size", 4 * d["d_model"]),
                      num_local_experts=ffn.get("moe_num_experts", 0), num_experts_per_tok=ffn.get("moe_top_k", 0),
                      rope_theta=attn.get("rope_theta", 10000.0), norm_type="layernorm_nobias", clip_qkv=attn.get("clip_qkv"),
                      max_position_embeddings=d.get("max_seq_len", 2048))
        kw["model_type"] = mt
        kw["extra"] = extra
        return cls(**kw)

    @classmethod
    def from_pretrained(cls, path: str) -> "ModelConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> Dict[str, Any]:
        d = dataclasses.asdict(self)
        d.update(d.pop("extra"))
        return d


@dataclass
class MixerDesign:
    """What a layer-by-layer design fixes itself; everything else comes from its config.json.  `constants` gives ModelConfig fields from
    the config; `mixers` holds what a kind of mixer has in this design, under the sizes that the config gives."""
    constants: Callable[[Dict[str, Any]], Dict[str, Any]]
    feed_forwards: Tuple[str, ...]
    gated: bool = True
    moe: Dict[str, Any] = field(default_factory=dict)
    mixers: Dict[str, Dict[str, Any]] = field(default_factory=dict)
    dense_act: str = ""


def _vabunex_constants(d: Dict[str, Any]) -> Dict[str, Any]:
    return dict(layer_style="parallel", parallel_residual=True, hidden_act="gelu_tanh", norm_weight_offset=1.0,
                embedding_multiplier=float(d["embedding"]["scale"]), max_position_embeddings=int(d.get("max_position_embeddings", 1 << 20)))


def _sapudra_constants(d: Dict[str, Any]) -> Dict[str, Any]:
    cap = d.get("logit_softcap")
    return dict(layer_style="post", norm_type="layernorm", hidden_act="relu2", residual_multiplier=float(d["residual_mult"]),
                learned_positions=True, max_position_embeddings=int(d["max_positions"]),
                final_logit_softcapping=float(cap) if cap is not None else None)


def _saredra_constants(d: Dict[str, Any]) -> Dict[str, Any]:
    return dict(layer_style="pre", hidden_act="silu", max_position_embeddings=int(d.get("max_position_embeddings", 1 << 20)))


def _fegolorn_constants(d: Dict[str, Any]) -> Dict[str, Any]:
    cap, bigram = d.get("logit_softcap"), d["embedding"].get("bigram")
    return dict(layer_style="sandwich", residual_gate=True, layer_scale=True, norm_scalar=True, hidden_act="silu",
                embedding_multiplier=float(d["embedding"]["scale"]), final_logit_softcapping=float(cap) if cap is not None else None,
                bigram=tuple(int(bigram[n]) for n in ("buckets", "mul_prev", "mul_cur")) if bigram else None,
                max_position_embeddings=int(d.get("max_position_embeddings", 1 << 20)))


_MIXER_DESIGNS = {
    "vabunex": MixerDesign(_vabunex_constants, ("dense",)),
    "sapudra": MixerDesign(_sapudra_constants, ("dense", "moe"), gated=False, mixers={"attention": dict(qk_norm=True)}),
    "saredra": MixerDesign(_saredra_constants, ("dense", "moe"), moe=dict(score="softmax", renorm=False, group_top=1),
                           mixers={"attention": dict(sink="unit", gate=True),
                                   "parallel": dict(left=dict(type="attention", bias=True, sink="learned"), right=dict(type="mamba2"))}),
    "fegolorn": MixerDesign(_fegolorn_constants, ("dense", "moe"), moe=dict(score="softmax", bias=True, shared_gate=False), dense_act="clamped_swiglu",
                            mixers={"attention": dict(qk_norm=True, rot_values=True),
                                    "latent_attention": dict(gate="element", rot_layout="halves")}),
}


def _moe_spec(mlp: Dict[str, Any], design: MixerDesign) -> MoeSpec:
    r, groups, shared = mlp["router"], mlp["router"].get("groups"), mlp.get("shared")
    return MoeSpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(mlp["expert"]["ff"]), scale=float(r.get("scale", 1.0)),
                   groups=int(groups["count"]) if groups else 0, keep=int(groups["keep"]) if groups else 0,
                   shared_ff=int(shared["ff"]) if shared else 0, gated=design.gated, **design.moe)


def _mixer_params(own: Dict[str, Any], fixed: Dict[str, Any]) -> Dict[str, Any]:
    """A mixer's sizes from the config over what the design fixes; mixers within a mixer likewise."""
    return {**{k: v for k, v in fixed.items() if not isinstance(v, dict)}, **own,
            **{k: _mixer_params(own[k], v) for k, v in fixed.items() if isinstance(v, dict)}}


def _owner(i: int, specs: List[LayerSpec]) -> int:
    """The layer whose tensors layer i uses, through others that have none of their own."""
    j, seen = i, set()
    while specs[j].weights_of is not None:
        seen.add(j)
        j = specs[j].weights_of
        if not 0 <= j < len(specs) or j in seen:
            raise ValueError(f"layer {i} uses the weights of layer {j}, which has none of its own")
    if dataclasses.replace(specs[i], weights_of=None) != specs[j]:
        raise ValueError(f"layer {i} uses the weights of layer {j}, which is of another kind or size")
    return j


def _mixer_model_kwargs(mt: str, d: Dict[str, Any]) -> Dict[str, Any]:
    """ModelConfig fields of a config.json that lists its layers (`layers`, `loop`, `norm`, `vocab`, `width`)."""
    design = _MIXER_DESIGNS[mt]
    specs = []
    for i, layer in enumerate(d["layers"]):
        mlp = layer.get("mlp")
        kind = mlp.get("kind", "dense") if mlp is not None else None
        if kind is not None and kind not in design.feed_forwards:
            raise NotImplementedError(f"layer {i}: feed-forward kind {kind!r}")
        specs.append(LayerSpec(layer["type"], _mixer_params(layer["mixer"], design.mixers.get(layer["type"], {})),
                               int(mlp["ff"]) if kind == "dense" else 0, _moe_spec(mlp, design) if kind == "moe" else None, design.gated,
                               design.dense_act if kind == "dense" else "", float(mlp["limit"]) if kind == "dense" and design.dense_act else 0.0,
                               int(layer["weights_of"]) if layer.get("weights_of") is not None else None))
    owners = [_owner(i, specs) for i in range(len(specs))]
    for i, j in enumerate(owners):
        specs[i].weights_of = j if j != i else None
    loop = d.get("loop")
    if loop is not None:
        loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not (0 <= loop[0] <= loop[1] <= len(specs)) or loop[2] < 0:
            raise ValueError(f"loop {loop} does not fit {len(specs)} layers")
    flat = [p for s in specs for p in ([s.params] if "heads" in s.params else [v for v in s.params.values() if isinstance(v, dict)])]
    most = lambda name: max([int(p[name]) for p in flat if name in p] + [1])
    return dict(dict(model_type=mt, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), intermediate_size=max([s.ff for s in specs] + [1]),
                     num_hidden_layers=len(specs), num_attention_heads=most("heads"),
                     num_key_value_heads=most("kv_heads" if any("kv_heads" in p for p in flat) else "heads"),
                     head_dim=most("dim"), rms_norm_eps=float(d["norm"]["eps"]), layer_specs=specs,
                     layer_loop=loop, eos_token_id=d.get("eos_token_id"), bos_token_id=d.get("bos_token_id"),
                     torch_dtype=d.get("torch_dtype", "bfloat16"), extra={}), **design.constants(d))


def mistral_7b() -> ModelConfig:
    """Mistral-7B-v0.1 architecture (the headline benchmark model)."""
    return ModelConfig(model_type="mistral", vocab_size=32000, hidden_size=4096, intermediate_size=14336,
                       num_hidden_layers=32, num_attention_heads=32, num_key_value_heads=8, head_dim=128,
                       rms_norm_eps=1e-5, rope_theta=10000.0, max_position_embeddings=32768, sliding_window=4096)


def llama3_8b() -> ModelConfig:
    return ModelConfig(model_type="llama", vocab_size=128256, hidden_size=4096, intermediate_size=14336,
                       num_hidden_layers=32, num_attention_heads=32, num_key_value_heads=8, head_dim=128,
                       rms_norm_eps=1e-5, rope_theta=500000.0, max_position_embeddings=8192)


def llama3_70b() -> ModelConfig:
    return ModelConfig(model_type="llama", vocab_size=128256, hidden_size=8192, intermediate_size=28672,
                       num_hidden_layers=80, num_attention_heads=64, num_key_value_heads=8, head_dim=128,
                       rms_norm_eps=1e-5, rope_theta=500000.0, max_position_embeddings=8192)


def mixtral_8x7b() -> ModelConfig:
    return ModelConfig(model_type="mixtral", vocab_size=32000, hidden_size=4096, intermediate_size=14336,
                       num_hidden_layers=32, num_attention_heads=32, num_key_value_heads=8, head_dim=128,
                       rms_norm_eps=1e-5, rope_theta=1e6, max_position_embeddings=32768,
                       num_local_experts=8, num_experts_per_tok=2)


def tiny_llama(vocab_size: int = 32000) -> ModelConfig:
    """The CPU plumbing model: 2 layers, hidden 256, 4 heads, 2 KV heads, intermediate 688."""
    return ModelConfig(model_type="llama", vocab_size=vocab_size, hidden_size=256, intermediate_size=688,
                       num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2, head_dim=64,
                       rms_norm_eps=1e-5, rope_theta=10000.0, max_position_embeddings=2048, torch_dtype="float32")


def _env(name: str, default, cast=None):
    v = os.environ.get(name)
    if v is None or v == "":
        return default
    if cast is bool:
        return v.lower() in ("1", "true", "yes", "on")
    return (cast or type(default))(v)


@dataclass
class EngineConfig:
    """Serving knobs.  Defaults follow `launcher/src/main.rs:413-560` of the reference."""

    model_id: str = ""
    revision: Optional[str] = None
    source: str = "hub"
    adapter_source: str = "hub"
    default_adapter_source: Optional[str] = None
    dtype: Optional[str] = None
    quantize: Optional[str] = None
    kv_cache_dtype: Optional[str] = None            # "fp8": e4m3 pages with per-layer k / v scales (None: the model's dtype)
    num_shard: int = 1
    max_concurrent_requests: int = 1024
    max_best_of: int = 2
    max_stop_sequences: int = 4
    max_input_length: int = 1024
    max_total_tokens: int = 2048
    max_batch_prefill_tokens: int = 4096
    max_batch_total_tokens: Optional[int] = None
    waiting_served_ratio: float = 1.2
    max_waiting_tokens: int = 20
    # in-process engine, saturated queue: let this many rows drain (for at most that many decode steps) before new prompts
    # interrupt the running batch, so that one prefill pass serves several prompts and most steps stay pure decode graphs
    prefill_min_rows: int = 8
    prefill_max_wait_steps: int = 8
    max_active_adapters: int = 1024
    adapter_cycle_time_s: int = 2
    adapter_memory_fraction: float = 0.1
    eager_prefill: bool = True
    prefix_caching: bool = False
    chunked_prefill: bool = False
    speculative_tokens: int = 0
    speculation_max_batch_size: int = 32
    compile: bool = True                      # CUDA-graph the decode step
    compile_max_batch_size: int = 256
    compile_max_rank: int = 64
    cuda_memory_fraction: float = 1.0
    memory_wiggle_room: float = 0.9
    block_size: int = 32                      # KV page size in tokens
    host_adapter_cache_gb: float = 16.0       # pinned host tier for adapter exchange
    preloaded_adapter_ids: List[str] = field(default_factory=list)
    preloaded_adapter_source: Optional[str] = None
    merge_adapter_weights: bool = False
    port: int = 3000
    hostname: str = "0.0.0.0"
    shard_uds_path: str = "/tmp/lorax-server"
    master_addr: str = "127.0.0.1"
    master_port: int = 29500
    otlp_endpoint: Optional[str] = None
    json_output: bool = False
    cors_allow_origin: List[str] = field(default_factory=list)
    watermark_gamma: float = 0.5
    watermark_delta: float = 2.0
    profiler_dir: Optional[str] = None
    tokenizer_config_path: Optional[str] = None
    fused_collectives: bool = True            # in-kernel NVLink collectives (False = NCCL baseline mode)

    @classmethod
    def from_env(cls, **overrides) -> "EngineConfig":
        c = cls()
        c.model_id = _env("MODEL_ID", c.model_id)
        c.num_shard = _env("NUM_SHARD", c.num_shard)
        c.quantize = _env("QUANTIZE", c.quantize, str)
        c.kv_cache_dtype = _env("KV_CACHE_DTYPE", c.kv_cache_dtype, str)
        c.dtype = _env("DTYPE", c.dtype, str)
        c.max_input_length = _env("MAX_INPUT_LENGTH", c.max_input_length)
        c.max_total_tokens = _env("MAX_TOTAL_TOKENS", c.max_total_tokens)
        c.max_batch_prefill_tokens = _env("MAX_BATCH_PREFILL_TOKENS", c.max_batch_prefill_tokens)
        c.max_batch_total_tokens = _env("MAX_BATCH_TOTAL_TOKENS", c.max_batch_total_tokens, int)
        c.waiting_served_ratio = _env("WAITING_SERVED_RATIO", c.waiting_served_ratio)
        c.max_waiting_tokens = _env("MAX_WAITING_TOKENS", c.max_waiting_tokens)
        c.max_active_adapters = _env("MAX_ACTIVE_ADAPTERS", c.max_active_adapters)
        c.adapter_cycle_time_s = _env("ADAPTER_CYCLE_TIME_S", c.adapter_cycle_time_s)
        c.adapter_memory_fraction = _env("ADAPTER_MEMORY_FRACTION", c.adapter_memory_fraction)
        c.prefix_caching = _env("PREFIX_CACHING", c.prefix_caching, bool)
        c.chunked_prefill = _env("CHUNKED_PREFILL", c.chunked_prefill, bool)
        c.speculative_tokens = _env("SPECULATIVE_TOKENS", c.speculative_tokens)
        c.speculation_max_batch_size = _env("LORAX_SPECULATION_MAX_BATCH_SIZE", c.speculation_max_batch_size)
        c.compile = _env("LORAX_COMPILE", c.compile, bool)
        c.compile_max_batch_size = _env("LORAX_COMPILE_MAX_BATCH_SIZE", c.compile_max_batch_size)
        c.compile_max_rank = _env("LORAX_COMPILE_MAX_RANK", c.compile_max_rank)
        c.cuda_memory_fraction = _env("CUDA_MEMORY_FRACTION", c.cuda_memory_fraction)
        c.memory_wiggle_room = _env("MEMORY_WIGGLE_ROOM", c.memory_wiggle_room)
        c.watermark_gamma = _env("WATERMARK_GAMMA", c.watermark_gamma)
        c.watermark_delta = _env("WATERMARK_DELTA", c.watermark_delta)
        c.profiler_dir = _env("LORAX_PROFILER_DIR", c.profiler_dir, str)
        c.master_addr = _env("MASTER_ADDR", c.master_addr)
        c.master_port = _env("MASTER_PORT", c.master_port)
        c.port = _env("PORT", c.port)
        for k, v in overrides.items():
            if v is not None:
                if not hasattr(c, k):
                    raise KeyError(f"unknown engine option {k!r}")
                setattr(c, k, v)
        return c
