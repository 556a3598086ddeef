"""Typed configuration of the engine.

``ModelConfig`` is built from a HuggingFace-style ``config.json`` dict (or one of
the named architecture presets used by the benchmarks), the remaining classes
mirror the knobs the reference exposes through vLLM's ``EngineArgs`` and its
``additional_config`` dictionary (vllm_gcu/gcu.py:184-354).
"""
from __future__ import annotations

import dataclasses
import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import Any, Optional

import torch

_DTYPES = {"bfloat16": torch.bfloat16, "float16": torch.float16, "float32": torch.float32,
           "bf16": torch.bfloat16, "fp16": torch.float16, "fp32": torch.float32,
           "half": torch.float16, "float": torch.float32}


def to_dtype(x: Any) -> torch.dtype:
    if isinstance(x, torch.dtype):
        return x
    return _DTYPES[str(x).replace("torch.", "")]


@dataclass(frozen=True)
class AttentionSpec:
    """Attention over cached keys and values (layers/key_attention.py)."""
    num_heads: int
    num_kv_heads: int
    head_dim: int
    scale: float                           # score scale
    rot_dims: int = 0                      # rotated dimensions of every head
    rot_base: float = 10000.0
    v_head_dim: int = 0                    # 0: the keys are their own values
    softcap: float = 0.0                   # scores become softcap * tanh(score / softcap); 0: none
    chunk: int = 0                         # keys of the query's own chunk of positions; 0: all
    window: int = 0                        # the last keys up to the query; 0: all
    # what follows is read by GroupedAttention
    rot_halves: bool = False               # dimension i turns with i + rot_dims / 2, not neighbours
    # YaRN: factor, original length, turns of the fast and of the slow end of the ramp
    rot_scaling: tuple[float, ...] = ()
    qk_norm: bool = False                  # norms over the whole query and key projections
    v_norm: bool = False                   # values divided by their root mean square, per head
    v_mix: bool = False                    # values mixed with those of the first such layer
    sink: str = ""                         # "learnt" score per head, "zero" (1 joins the sum), none
    distance_bias: bool = False            # a slope per head times the distance comes off the score
    # queries times 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1) at position p
    temp_coef: float = 0.0
    temp_every: int = 1

    @property
    def cached_per_token(self) -> int:
        return self.num_kv_heads * (self.head_dim + (self.v_head_dim or self.head_dim))


@dataclass(frozen=True)
class MemorySpec:
    """Matrix memory with exponential gates (layers/recurrent.py)."""
    num_heads: int
    head_dim: int
    v_head_dim: int
    gate_cap: float                        # soft cap of the gates' projections


@dataclass(frozen=True)
class DeltaSpec:
    """Gated delta rule with one decay per key channel (layers/recurrent.py)."""
    num_heads: int
    num_kv_heads: int                      # query / key heads
    head_dim: int
    v_head_dim: int
    conv_taps: int
    decay_rank: int                        # inner width of the decay's two-step projection
    gate_rank: int                         # and of the output gate's


@dataclass(frozen=True)
class TimeMixSpec:
    """Linear recurrence with one decay per head and key channel and a bonus for the current token
    (layers/recurrent.py)."""
    num_heads: int
    head_dim: int                          # keys and values
    decay_rank: int                        # inner width of the decay's two-step projection


@dataclass(frozen=True)
class LayerSpec:
    """One layer of a design whose layers differ: mixer type and sizes, feed-forward sizes."""
    mixer: str                             # "latent_attention", or with ``parts`` any name
    num_heads: int = 0
    head_dim: int = 0                      # query / key dimensions per head
    v_head_dim: int = 0
    kv_lora_rank: int = 0                  # latent width
    scale: float = 1.0                     # score scale
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    intermediate_size: int = 0             # dense feed-forward
    shared_intermediate_size: int = 0      # shared expert beside the routed ones
    router_scale: float = 1.0              # factor of the routing weights
    router_groups: int = 1                 # groups of neighbouring experts
    router_keep: int = 1                   # groups a token's experts come from
    rot_dim: int = 0                       # latent attention: rotated query / key dimensions
    rot_base: float = 10000.0
    sink: bool = False                     # latent attention: learnt term in the denominator
    head_gate: bool = False                # latent attention: one gate per head, not per channel
    # mixer as a sum of parts: (checkpoint prefix, factor, spec)
    parts: tuple[tuple[str, float, Any], ...] = ()

    @property
    def has_mlp(self) -> bool:
        return self.num_experts > 0 or self.intermediate_size > 0

    @property
    def cached_per_token(self) -> int:
        """Elements a token leaves in the paged cache."""
        return self.kv_lora_rank + self.rot_dim + sum(
            s.cached_per_token for _, _, s in self.parts if isinstance(s, AttentionSpec))


@dataclass
class ModelConfig:
    architecture: str = "LlamaForCausalLM"
    vocab_size: int = 32000
    hidden_size: int = 4096
    intermediate_size: int = 11008
    num_hidden_layers: int = 32
    num_attention_heads: int = 32
    num_key_value_heads: int = 32
    head_dim: int = 0                      # 0 -> hidden_size // num_attention_heads
    rms_norm_eps: float = 1e-6
    rope_theta: float = 10000.0
    rope_scaling: Optional[dict] = None
    partial_rotary_factor: float = 1.0
    rope_is_neox: bool = True
    max_position_embeddings: int = 8192
    tie_word_embeddings: bool = False
    attention_bias: bool = False
    mlp_bias: bool = False
    hidden_act: str = "silu"
    qk_norm: bool = False                  # per-head RMSNorm on q and k (Qwen3)
    sandwich_norm: bool = False            # GLM-4-0414: extra post-attn / post-mlp norms
    sliding_window: int = 0
    dtype: torch.dtype = torch.bfloat16
    # MoE
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    num_shared_experts: int = 0
    first_k_dense_replace: int = 0
    moe_layer_freq: int = 1
    norm_topk_prob: bool = True
    scoring_func: str = "softmax"
    n_group: int = 1
    topk_group: int = 1
    routed_scaling_factor: float = 1.0
    topk_method: str = "greedy"            # "noaux_tc" adds e_score_correction_bias
    # MLA
    q_lora_rank: int = 0
    kv_lora_rank: int = 0
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    # MTP
    num_nextn_predict_layers: int = 0
    # quantisation (HF quantization_config / quantize_config.json, see layers/quant)
    quantization: Optional[str] = None
    quant_config: Optional[dict] = None
    kv_cache_dtype: str = "auto"
    # designs described layer by layer (None: every layer has the sizes above)
    layer_specs: Optional[tuple[LayerSpec, ...]] = None
    residual_alpha: float = 1.0            # norm after the sum: norm(alpha * x + sublayer(x))
    residual_mult: float = 1.0             # norm in front: x + residual_mult * sublayer(norm(x))
    norm_groups: int = 1                   # parts of a row that are normalised each for itself
    conv_taps: int = 0                     # causal convolution in front of every mixer; 0: none
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    # (start, stop, times): layers start .. stop - 1 run that often in a row, same weights
    loop: Optional[tuple[int, int, int]] = None
    extra: dict = field(default_factory=dict)

    def __post_init__(self) -> None:
        self.dtype = to_dtype(self.dtype)
        if self.layer_specs is not None and len(self.layer_specs) != self.num_hidden_layers:
            # a shorter or longer model of the same layers
            n = self.num_hidden_layers
            reps = -(-n // len(self.layer_specs))
            self.layer_specs = (tuple(self.layer_specs) * reps)[:n]
        if self.loop is not None:
            start, stop, times = self.loop
            stop = min(stop, self.num_hidden_layers)
            self.loop = (start, stop, times) if start < stop else None
        if self.head_dim <= 0:
            self.head_dim = self.hidden_size // self.num_attention_heads

    # -- derived ---------------------------------------------------------
    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank > 0

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def rotary_dim(self) -> int:
        d = self.qk_rope_head_dim if self.is_mla else self.head_dim
        return int(d * self.partial_rotary_factor)

    @property
    def layer_runs(self) -> list[tuple[int, Optional[int]]]:
        """``(layer, pass)`` in the order of execution; ``pass`` is the number of the loop's pass
        whose first layer this is, else None.  Every run has a cache of its own."""
        n = self.num_hidden_layers
        start, stop, times = self.loop or (0, 0, 0)
        return [(i, None) for i in range(start)] + \
            [(i, t if i == start else None) for t in range(times) for i in range(start, stop)] + \
            [(i, None) for i in range(stop, n)]

    def is_moe_layer(self, layer_idx: int) -> bool:
        if not self.is_moe or layer_idx < self.first_k_dense_replace \
                or layer_idx % self.moe_layer_freq != 0:
            return False
        # Qwen MoE configs: dense layers listed by index, experts on every n-th layer
        if layer_idx in (self.extra.get("mlp_only_layers") or ()):
            return False
        step = int(self.extra.get("decoder_sparse_step") or 1)
        return (layer_idx + 1) % step == 0

    def kv_bytes_per_token(self, tp_size: int = 1) -> int:
        es = 1 if self.kv_cache_dtype.startswith("fp8") or self.kv_cache_dtype == "int8" else \
            torch.empty((), dtype=self.dtype).element_size()
        if self.layer_specs is not None:
            return sum(self.layer_specs[i].cached_per_token for i, _ in self.layer_runs) * es
        if self.is_mla:
            return self.num_hidden_layers * (self.kv_lora_rank + self.qk_rope_head_dim) * es
        kvh = max(1, self.num_key_value_heads // tp_size)
        return self.num_hidden_layers * 2 * kvh * self.head_dim * es

    def window_for_layer(self, layer_idx: int) -> int:
        """Sliding-window length of one layer (0 = full attention).  Checkpoints name the
        layers that use the window by ``layer_types``, or by ``use_sliding_window`` with
        ``max_window_layers`` (Qwen2: the layers from that index on); a ``sliding_window`` value
        next to ``use_sliding_window: false`` is not in force."""
        w = int(self.sliding_window or 0)
        if w <= 0:
            return 0
        types = self.extra.get("layer_types")
        if isinstance(types, (list, tuple)) and layer_idx < len(types):
            return w if "sliding" in str(types[layer_idx]) else 0
        use = self.extra.get("use_sliding_window")
        if use is False:
            return 0
        if use is True and self.extra.get("max_window_layers") is not None:
            return w if layer_idx >= int(self.extra["max_window_layers"]) else 0
        return w

    @property
    def eos_token_ids(self) -> tuple[int, ...]:
        """End-of-sequence ids of the checkpoint (``eos_token_id`` of ``config.json``, an int or
        a list, plus those of ``generation_config.json``); empty for architecture presets."""
        out: list[int] = []
        for src in (self.extra.get("eos_token_id"), self.extra.get("generation_eos_token_id")):
            for t in (src if isinstance(src, (list, tuple)) else [src]):
                if isinstance(t, int) and t >= 0 and t not in out:
                    out.append(t)
        return tuple(out)

    @property
    def eos_token_id(self) -> Optional[int]:
        ids = self.eos_token_ids
        return ids[0] if ids else None

    # -- construction ----------------------------------------------------
    @classmethod
    def from_hf_dict(cls, d: dict, **overrides) -> "ModelConfig":
        if d.get("architecture") == "Sapapel" or "SapapelForCausalLM" in (
                d.get("architectures") or ()):
            return cls._from_layer_list(d, **overrides)
        if d.get("architecture") == "Fizunex" or "FizunexForCausalLM" in (
                d.get("architectures") or ()):
            return cls._from_mixer_list(d, **overrides)
        if d.get("architecture") == "Fepopel" or "FepopelForCausalLM" in (
                d.get("architectures") or ()):
            return cls._from_looped_list(d, **overrides)
        if d.get("architecture") == "Vadelix" or "VadelixForCausalLM" in (
                d.get("architectures") or ()):
            return cls._from_prenorm_list(d, **overrides)
        archs = d.get("architectures") or ["LlamaForCausalLM"]
        for nested in ("text_config", "language_config", "llm_config"):
            if isinstance(d.get(nested), dict):
                # multimodal configs nest the language model's fields; vision_config, token
                # ids and everything else stay reachable through ``extra``
                inner_arch = (d[nested].get("architectures") or [None])[0]
                d = {**{k: v for k, v in d.items() if k != nested},
                     "llm_architecture": inner_arch, "llm_model_type": d[nested].get("model_type"),
                     **{k: v for k, v in d[nested].items()
                        if k not in ("architectures", "model_type")}}
        if archs[0] == "GPTBigCodeForCausalLM":
            # GPT-2 style field names; multi-query attention = one key / value head
            d = dict(d)
            heads = d["n_head"]
            d.setdefault("hidden_size", d["n_embd"])
            d.setdefault("num_hidden_layers", d["n_layer"])
            d.setdefault("num_attention_heads", heads)
            d.setdefault("num_key_value_heads", 1 if d.get("multi_query", True) else heads)
            d.setdefault("intermediate_size", d.get("n_inner") or 4 * d["n_embd"])
            d.setdefault("max_position_embeddings", d.get("n_positions", 8192))
            d.setdefault("rms_norm_eps", d.get("layer_norm_epsilon", 1e-5))
            d.setdefault("hidden_act", d.get("activation_function", "gelu_pytorch_tanh"))
            d.setdefault("head_dim", d["n_embd"] // heads)
            d["tie_word_embeddings"] = True
            d["attention_bias"] = True
        if archs[0] in ("ChatGLMModel", "ChatGLMForConditionalGeneration"):
            # ChatGLM2 / 3 / GLM-4-9B configs use their own field names
            d = dict(d)
            heads = d["num_attention_heads"]
            d.setdefault("num_hidden_layers", d.get("num_layers"))
            d.setdefault("intermediate_size", d.get("ffn_hidden_size"))
            d.setdefault("num_key_value_heads",
                         d.get("multi_query_group_num", heads) if d.get("multi_query_attention")
                         else heads)
            d.setdefault("head_dim", d.get("kv_channels", d["hidden_size"] // heads))
            d.setdefault("rms_norm_eps", d.get("layernorm_epsilon", 1e-5))
            d.setdefault("vocab_size", d.get("padded_vocab_size"))
            d.setdefault("max_position_embeddings", d.get("seq_length", 8192))
            d.setdefault("attention_bias", bool(d.get("add_qkv_bias", False)))
            d.setdefault("rope_theta", 10000.0 * float(d.get("rope_ratio", 1.0)))
            d.setdefault("tie_word_embeddings", False)
        names = {f.name for f in dataclasses.fields(cls)}
        kw: dict[str, Any] = {"architecture": archs[0]}
        alias = {"n_routed_experts": "num_experts", "num_local_experts": "num_experts",
                 "n_shared_experts": "num_shared_experts", "torch_dtype": "dtype"}
        extra = {}
        for k, v in d.items():
            k2 = alias.get(k, k)
            if k2 in names and v is not None:
                kw[k2] = v
            else:
                extra[k] = v
        arch = archs[0]
        if "Qwen3" in arch:
            kw.setdefault("qk_norm", True)
        if arch.startswith("Glm4"):
            kw.setdefault("sandwich_norm", True)
            kw.setdefault("rope_is_neox", False)
            kw.setdefault("partial_rotary_factor", d.get("partial_rotary_factor", 0.5))
        if "Deepseek" in arch:
            kw.setdefault("rope_is_neox", False)
        if arch in ("DeepseekV3ForCausalLM", "DeepSeekMTPModel") or \
                d.get("model_type") == "deepseek_v3":
            # configs written by newer libraries leave the V3 routing to the model type:
            # sigmoid scores, group-limited top-k with a learnt selection bias
            kw.setdefault("scoring_func", "sigmoid")
            kw.setdefault("topk_method", "noaux_tc")
        if arch.startswith("ChatGLM"):
            kw.setdefault("rope_is_neox", False)
            kw.setdefault("partial_rotary_factor", 0.5)
        if "rope_parameters" in d and isinstance(d["rope_parameters"], dict):
            rp = d["rope_parameters"]
            kw.setdefault("rope_theta", rp.get("rope_theta", kw.get("rope_theta", 10000.0)))
            if kw.get("rope_scaling") is None and (rp.get("mrope_section") or
                                                   rp.get("rope_type", "default") != "default"):
                kw["rope_scaling"] = rp
        qc = d.get("quantization_config")
        if qc:
            kw["quant_config"] = qc
            kw["quantization"] = qc.get("quant_method")
        kw["extra"] = extra
        kw.update(overrides)
        return cls(**kw)

    @classmethod
    def _from_layer_list(cls, d: dict, **overrides) -> "ModelConfig":
        """Sapapel's ``config.json``: ``vocab``, ``width``, ``norm.eps``, ``postln_alpha`` and one
        entry of ``layers`` per layer with its mixer's and its feed-forward's sizes."""
        specs = []
        for i, layer in enumerate(d["layers"]):
            if layer["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
            m, f = layer["mixer"], layer.get("mlp")
            moe = {}
            if f is not None:
                if f.get("kind", "moe") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
                moe = dict(num_experts=int(f["router"]["experts"]),
                           num_experts_per_tok=int(f["router"]["top"]),
                           moe_intermediate_size=int(f["expert"]["ff"]))
                if not 0 < moe["num_experts_per_tok"] <= moe["num_experts"]:
                    raise ValueError(f"layer {i}: {moe['num_experts_per_tok']} of "
                                     f"{moe['num_experts']} experts per token")
            specs.append(LayerSpec("latent_attention", int(m["heads"]), int(m["dim"]),
                                   int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]), **moe))
        if not specs:
            raise ValueError("the configuration lists no layers")
        kw: dict[str, Any] = dict(
            architecture="SapapelForCausalLM", vocab_size=int(d["vocab"]),
            hidden_size=int(d["width"]), num_hidden_layers=len(specs),
            rms_norm_eps=float(d["norm"]["eps"]), residual_alpha=float(d["postln_alpha"]),
            layer_specs=tuple(specs),
            # the largest layer stands for the model where one number is asked for
            num_attention_heads=max(s.num_heads for s in specs), num_key_value_heads=1,
            head_dim=max(s.head_dim for s in specs),
            v_head_dim=max(s.v_head_dim for s in specs),
            kv_lora_rank=max(s.kv_lora_rank for s in specs),
            num_experts=max(s.num_experts for s in specs),
            num_experts_per_tok=max(s.num_experts_per_tok for s in specs),
            moe_intermediate_size=max(s.moe_intermediate_size for s in specs),
            scoring_func="sigmoid", norm_topk_prob=False,
            # no positions in the design, so no limit of its own: bounds the block tables only
            max_position_embeddings=int(d.get("max_position_embeddings", 131072)),
            extra={k: v for k, v in d.items() if k not in (
                "layers", "vocab", "width", "norm", "postln_alpha", "architecture",
                "architectures", "max_position_embeddings")})
        kw.update(overrides)
        return cls(**kw)

    @classmethod
    def _from_mixer_list(cls, d: dict, **overrides) -> "ModelConfig":
        """Fizunex's ``config.json``: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``,
        ``logit_scale`` and one entry of ``layers`` per layer.  The inner widths of a delta layer's
        two-step projections are no numbers of the file: a checkpoint's tensors give them
        (``tensor_shapes``), else ``decay_rank`` / ``gate_rank`` of the mixer, else its ``dim``."""
        shapes = overrides.pop("tensor_shapes", None) or {}
        specs = []
        for i, layer in enumerate(d["layers"]):
            m, f, where = layer["mixer"], layer.get("mlp"), f"layer {i}"
            ff = 0
            if f is not None:
                if f.get("kind", "dense") != "dense":
                    raise ValueError(f"{where}: unknown feed-forward {f['kind']!r}")
                ff = int(f["ff"])
            if layer["type"] == "channel_delta":
                def rank(tensor: str, key: str) -> int:
                    s = shapes.get(f"l{i}.mix.{tensor}")
                    return int(s[0] if s is not None else m.get(key) or m["dim"])
                parts = (("", 1.0, DeltaSpec(
                    int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]),
                    int(m["conv"]), rank("a1", "decay_rank"), rank("g1", "gate_rank"))),)
            elif layer["type"] == "parallel":
                a, b = m["left"], m["right"]
                if int(a.get("vdim", a["dim"])) != int(a["dim"]):
                    raise ValueError(f"{where}: values are the keys, so {a['vdim']} value "
                                     f"dimensions cannot differ from {a['dim']} key dimensions")
                parts = (("left.", float(m["left_scale"]), AttentionSpec(
                    int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), float(a["scale"]),
                    int(a["rot"]["dims"]), float(a["rot"]["base"]))),
                    ("right.", float(m["right_scale"]), MemorySpec(
                        int(b["heads"]), int(b["dim"]), int(b["vdim"]), float(b["gate_cap"]))))
            else:
                raise ValueError(f"{where}: unknown mixer {layer['type']!r}")
            specs.append(LayerSpec(layer["type"], intermediate_size=ff, parts=parts))
        if not specs:
            raise ValueError("the configuration lists no layers")
        attn = [s for sp in specs for _, _, s in sp.parts if isinstance(s, AttentionSpec)]
        kw: dict[str, Any] = dict(
            architecture="FizunexForCausalLM", vocab_size=int(d["vocab"]),
            hidden_size=int(d["width"]), num_hidden_layers=len(specs),
            rms_norm_eps=float(d["norm"]["eps"]), layer_specs=tuple(specs),
            embed_scale=float(d["embedding"]["scale"]), logit_scale=float(d["logit_scale"]),
            tie_word_embeddings=True,
            # the largest layer stands for the model where one number is asked for
            intermediate_size=max(s.intermediate_size for s in specs),
            num_attention_heads=max((s.num_heads for s in attn), default=1),
            num_key_value_heads=max((s.num_kv_heads for s in attn), default=1),
            head_dim=max((s.head_dim for s in attn), default=1),
            # no limit of the design's own: bounds the rotary and block tables only
            max_position_embeddings=int(d.get("max_position_embeddings", 131072)),
            extra={k: v for k, v in d.items() if k not in (
                "layers", "vocab", "width", "norm", "embedding", "logit_scale", "architecture",
                "architectures", "max_position_embeddings")})
        kw.update(overrides)
        return cls(**kw)

    @classmethod
    def _from_looped_list(cls, d: dict, **overrides) -> "ModelConfig":
        """Fepopel's ``config.json``: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``,
        ``loop`` and one entry of ``layers`` per layer with its mixer's and its feed-forward's
        sizes."""
        specs = []
        for i, layer in enumerate(d["layers"]):
            m, f, where = layer["mixer"], layer.get("mlp"), f"layer {i}"
            kw: dict[str, Any] = {}
            if f is not None and f.get("kind", "dense") == "dense":
                kw["intermediate_size"] = int(f["ff"])
            elif f is not None and f["kind"] == "moe":
                r, shared = f["router"], f.get("shared")
                kw.update(num_experts=int(r["experts"]), num_experts_per_tok=int(r["top"]),
                          router_scale=float(r.get("scale", 1.0)),
                          moe_intermediate_size=int(f["expert"]["ff"]),
                          shared_intermediate_size=int(shared["ff"]) if shared else 0)
                if not 0 < kw["num_experts_per_tok"] <= kw["num_experts"]:
                    raise ValueError(f"{where}: {kw['num_experts_per_tok']} of "
                                     f"{kw['num_experts']} experts per token")
            elif f is not None:
                raise ValueError(f"{where}: unknown feed-forward {f['kind']!r}")
            if layer["type"] == "latent_attention":
                rot = m.get("rot") or {}
                if int(rot.get("dims", m["rot_dim"])) != int(m["rot_dim"]):
                    raise ValueError(f"{where}: {rot['dims']} of {m['rot_dim']} dimensions rotated")
                specs.append(LayerSpec(
                    layer["type"], int(m["heads"]), int(m["dim"]), int(m["vdim"]),
                    int(m["kv_rank"]), float(m["scale"]), rot_dim=int(m["rot_dim"]),
                    rot_base=float(rot.get("base", 10000.0)), sink=True, head_gate=True, **kw))
            elif layer["type"] == "attention":
                specs.append(LayerSpec(layer["type"], parts=(("", 1.0, AttentionSpec(
                    int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), float(m["scale"]),
                    v_head_dim=int(m["vdim"]), softcap=float(m.get("softcap") or 0.0),
                    chunk=int((m.get("mask") or {}).get("size") or 0))),), **kw))
            else:
                raise ValueError(f"{where}: unknown mixer {layer['type']!r}")
        if not specs:
            raise ValueError("the configuration lists no layers")
        loop = d.get("loop")
        if loop:
            loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
            if not (0 <= loop[0] < loop[1] <= len(specs) and loop[2] > 0):
                raise ValueError(f"a loop over layers {loop[0]} to {loop[1]} of {len(specs)}, "
                                 f"{loop[2]} times")
        attn = [s for sp in specs for _, _, s in sp.parts]
        kw = dict(
            architecture="FepopelForCausalLM", vocab_size=int(d["vocab"]),
            hidden_size=int(d["width"]), num_hidden_layers=len(specs),
            rms_norm_eps=float(d["norm"]["eps"]), layer_specs=tuple(specs), loop=loop or None,
            embed_scale=float(d["embedding"]["scale"]),
            # the largest layer stands for the model where one number is asked for
            intermediate_size=max(s.intermediate_size for s in specs),
            num_attention_heads=max([s.num_heads for s in specs] + [s.num_heads for s in attn]),
            num_key_value_heads=max((s.num_kv_heads for s in attn), default=1),
            head_dim=max([s.head_dim + s.rot_dim for s in specs] + [s.head_dim for s in attn]),
            num_experts=max(s.num_experts for s in specs),
            num_experts_per_tok=max(s.num_experts_per_tok for s in specs),
            moe_intermediate_size=max(s.moe_intermediate_size for s in specs),
            # no limit of the design's own: bounds the rotary and block tables only
            max_position_embeddings=int(d.get("max_position_embeddings", 131072)),
            extra={k: v for k, v in d.items() if k not in (
                "layers", "vocab", "width", "norm", "embedding", "loop", "architecture",
                "architectures", "max_position_embeddings")})
        kw.update(overrides)
        return cls(**kw)

    @classmethod
    def _from_prenorm_list(cls, d: dict, **overrides) -> "ModelConfig":
        """Vadelix's ``config.json``: ``vocab``, ``width``, ``norm`` (eps, groups),
        ``residual_mult``, ``canon.taps`` and one entry of ``layers`` per layer.  The inner width of
        a decay's two-step projection is no number of the file: a checkpoint's tensors give it
        (``tensor_shapes``), else ``decay_rank`` of the mixer, else its ``dim``."""
        shapes = overrides.pop("tensor_shapes", None) or {}
        specs = []
        for i, layer in enumerate(d["layers"]):
            m, f, where = layer["mixer"], layer.get("mlp"), f"layer {i}"
            kw: dict[str, Any] = {}
            if f is not None and f.get("kind", "dense") == "dense":
                kw["intermediate_size"] = int(f["ff"])
            elif f is not None and f["kind"] == "moe":
                r, shared = f["router"], f.get("shared")
                groups = r.get("groups") or {"count": 1, "keep": 1}
                kw.update(num_experts=int(r["experts"]), num_experts_per_tok=int(r["top"]),
                          router_groups=int(groups["count"]), router_keep=int(groups["keep"]),
                          moe_intermediate_size=int(f["expert"]["ff"]),
                          shared_intermediate_size=int(shared["ff"]) if shared else 0)
                E, count, keep = kw["num_experts"], kw["router_groups"], kw["router_keep"]
                if E % count or not 0 < keep <= count:
                    raise ValueError(f"{where}: {keep} of {count} groups of {E} experts")
                if not 0 < kw["num_experts_per_tok"] <= E // count * keep:
                    raise ValueError(f"{where}: {kw['num_experts_per_tok']} of "
                                     f"{E // count * keep} experts per token")
            elif f is not None:
                raise ValueError(f"{where}: unknown feed-forward {f['kind']!r}")
            if layer["type"] == "wkv":
                rank = shapes.get(f"l{i}.mix.w1")
                spec: Any = TimeMixSpec(int(m["heads"]), int(m["dim"]), int(
                    rank[0] if rank is not None else m.get("decay_rank") or m["dim"]))
            elif layer["type"] in ("attention", "attention_2"):
                size = dict(num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]),
                            head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]),
                            scale=float(m["scale"]), v_mix=bool(m.get("v_mix")))
                if layer["type"] == "attention":
                    rot = m.get("rot") or {"dims": 0, "base": 1.0}
                    y = rot.get("scaling")
                    spec = AttentionSpec(
                        rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), rot_halves=True,
                        rot_scaling=tuple(float(y[k]) for k in ("factor", "original", "fast",
                                                                "slow")) if y else (),
                        qk_norm=True, v_norm=True, sink="learnt", **size)
                else:
                    t = m.get("q_temp") or {"coef": 0.0, "every": 1}
                    spec = AttentionSpec(
                        window=int((m.get("mask") or {}).get("size") or 0), distance_bias=True,
                        sink="zero", temp_coef=float(t["coef"]), temp_every=int(t["every"]), **size)
            else:
                raise ValueError(f"{where}: unknown mixer {layer['type']!r}")
            specs.append(LayerSpec(layer["type"], parts=(("", 1.0, spec),), **kw))
        if not specs:
            raise ValueError("the configuration lists no layers")
        H, groups = int(d["width"]), int(d["norm"].get("groups", 1))
        if H % groups:
            raise ValueError(f"a norm of {groups} groups over {H} coordinates")
        attn = [s for sp in specs for _, _, s in sp.parts if isinstance(s, AttentionSpec)]
        kw = dict(
            architecture="VadelixForCausalLM", vocab_size=int(d["vocab"]), hidden_size=H,
            num_hidden_layers=len(specs), layer_specs=tuple(specs),
            rms_norm_eps=float(d["norm"]["eps"]), norm_groups=groups,
            residual_mult=float(d.get("residual_mult", 1.0)),
            conv_taps=int(d["canon"]["taps"]), hidden_act="gelu_tanh",
            # the largest layer stands for the model where one number is asked for
            intermediate_size=max(s.intermediate_size for s in specs),
            num_attention_heads=max((s.num_heads for s in attn), default=1),
            num_key_value_heads=max((s.num_kv_heads for s in attn), default=1),
            head_dim=max((max(s.head_dim, s.v_head_dim) for s in attn), default=1),
            num_experts=max(s.num_experts for s in specs),
            num_experts_per_tok=max(s.num_experts_per_tok for s in specs),
            moe_intermediate_size=max(s.moe_intermediate_size for s in specs),
            # no limit of the design's own: bounds the rotary and block tables only
            max_position_embeddings=int(d.get("max_position_embeddings", 131072)),
            extra={k: v for k, v in d.items() if k not in (
                "layers", "vocab", "width", "norm", "canon", "residual_mult", "architecture",
                "architectures", "max_position_embeddings")})
        kw.update(overrides)
        return cls(**kw)

    @classmethod
    def from_pretrained(cls, path: str, **overrides) -> "ModelConfig":
        p = Path(path)
        d = json.loads((p / "config.json").read_text())
        if d.get("architecture") in ("Fizunex", "Vadelix"):
            from .utils.weights import tensor_shapes
            overrides = {"tensor_shapes": tensor_shapes(path), **overrides}
        cfg = cls.from_hf_dict(d, **overrides)
        gpath = p / "generation_config.json"
        if gpath.exists():
            try:
                gen = json.loads(gpath.read_text())
                cfg.extra["generation_eos_token_id"] = gen.get("eos_token_id")
                # sampling defaults the checkpoint recommends; the server applies them to
                # requests that leave the field out
                cfg.extra["generation_defaults"] = {
                    k: gen[k] for k in ("temperature", "top_p", "top_k", "repetition_penalty")
                    if gen.get(k) is not None and gen.get("do_sample", True)}
            except (OSError, ValueError):
                pass
        qpath = p / "quantize_config.json"
        if cfg.quant_config is None and qpath.exists():
            cfg.quant_config = json.loads(qpath.read_text())
            cfg.quantization = cfg.quantization or cfg.quant_config.get("quant_method")
        return cfg


def preset(name: str, **overrides) -> ModelConfig:
    """Architecture presets of the benchmark configurations (random-init weights)."""
    presets: dict[str, dict] = {
        "tiny-llama": dict(vocab_size=32000, hidden_size=256, intermediate_size=688,
                           num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2,
                           head_dim=64, rms_norm_eps=1e-6, rope_theta=10000.0,
                           max_position_embeddings=2048, dtype="float32"),
        "llama-3-8b": dict(vocab_size=128256, hidden_size=4096, intermediate_size=14336,
                           num_hidden_layers=32, num_attention_heads=32, num_key_value_heads=8,
                           head_dim=128, rms_norm_eps=1e-5, rope_theta=500000.0,
                           max_position_embeddings=8192, dtype="bfloat16"),
        "llama-3-70b": dict(vocab_size=128256, hidden_size=8192, intermediate_size=28672,
                            num_hidden_layers=80, num_attention_heads=64, num_key_value_heads=8,
                            head_dim=128, rms_norm_eps=1e-5, rope_theta=500000.0,
                            max_position_embeddings=8192, dtype="bfloat16"),
        "qwen3-30b-a3b": dict(architecture="Qwen3MoeForCausalLM", vocab_size=151936,
                              hidden_size=2048, intermediate_size=6144, num_hidden_layers=48,
                              num_attention_heads=32, num_key_value_heads=4, head_dim=128,
                              qk_norm=True, num_experts=128, num_experts_per_tok=8,
                              moe_intermediate_size=768, norm_topk_prob=True,
                              rms_norm_eps=1e-6, rope_theta=1000000.0,
                              max_position_embeddings=40960, dtype="bfloat16"),
        "deepseek-v3": dict(architecture="DeepseekV3ForCausalLM", vocab_size=129280,
                            hidden_size=7168, intermediate_size=18432, num_hidden_layers=61,
                            num_attention_heads=128, num_key_value_heads=128,
                            q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128,
                            qk_rope_head_dim=64, v_head_dim=128, head_dim=192,
                            num_experts=256, num_experts_per_tok=8, moe_intermediate_size=2048,
                            num_shared_experts=1, first_k_dense_replace=3, n_group=8,
                            topk_group=4, scoring_func="sigmoid", topk_method="noaux_tc",
                            routed_scaling_factor=2.5, norm_topk_prob=True,
                            num_nextn_predict_layers=1, rope_is_neox=False,
                            rms_norm_eps=1e-6, rope_theta=10000.0,
                            max_position_embeddings=163840, dtype="bfloat16"),
        "tiny-qwen3-moe": dict(architecture="Qwen3MoeForCausalLM", vocab_size=1024,
                               hidden_size=128, intermediate_size=256, num_hidden_layers=2,
                               num_attention_heads=4, num_key_value_heads=2, head_dim=32,
                               qk_norm=True, num_experts=8, num_experts_per_tok=2,
                               moe_intermediate_size=64, dtype="float32"),
        "tiny-deepseek": dict(architecture="DeepseekV3ForCausalLM", vocab_size=1024,
                              hidden_size=128, intermediate_size=256, num_hidden_layers=3,
                              num_attention_heads=4, num_key_value_heads=4, q_lora_rank=48,
                              kv_lora_rank=32, qk_nope_head_dim=16, qk_rope_head_dim=8,
                              v_head_dim=16, head_dim=24, num_experts=8, num_experts_per_tok=2,
                              moe_intermediate_size=32, num_shared_experts=1,
                              first_k_dense_replace=1, n_group=2, topk_group=1,
                              scoring_func="sigmoid", topk_method="noaux_tc",
                              routed_scaling_factor=2.5, num_nextn_predict_layers=1,
                              rope_is_neox=False, dtype="float32"),
    }
    if name in _LAYER_LIST_PRESETS:
        return ModelConfig.from_hf_dict(_LAYER_LIST_PRESETS[name], **overrides)
    kw = dict(presets[name])
    kw.update(overrides)
    return ModelConfig(**kw)


def _sapapel_preset(layers: int, vocab: int, width: int, heads: int, dim: int, vdim: int,
                    kv_rank: int, experts: int, top: int, ff: int) -> dict:
    layer = {"type": "latent_attention",
             "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank,
                       "scale": dim ** -0.5},
             "mlp": {"kind": "moe", "router": {"experts": experts, "top": top},
                     "expert": {"ff": ff}}}
    return {"architecture": "Sapapel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
            "postln_alpha": (2.0 * layers) ** 0.25, "layers": [layer] * layers}


def _fizunex_preset(pattern: str, vocab: int, width: int, ff: int, delta: dict, left: dict,
                    right: dict) -> dict:
    """``pattern``: one letter per layer, d for a gated delta layer, p for a parallel one."""
    mlp = {"kind": "dense", "ff": ff}
    kinds = {"d": {"type": "channel_delta", "mixer": delta, "mlp": mlp},
             "p": {"type": "parallel", "mlp": mlp,
                   "mixer": {"left": left, "right": right, "left_scale": 0.7, "right_scale": 0.7}}}
    return {"architecture": "Fizunex", "vocab": vocab, "width": width, "norm": {"eps": 1e-5},
            "embedding": {"scale": 1.0}, "logit_scale": 1.0, "layers": [kinds[c] for c in pattern]}


def _fizunex_mixers(heads: int, kv_heads: int, dim: int, memory_heads: int, memory_dim: int,
                    memory_vdim: int, conv: int = 4, rot_dims: int = 0) -> tuple[dict, dict, dict]:
    delta = {"heads": heads, "kv_heads": heads, "dim": dim, "vdim": dim, "conv": conv}
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
            "rot": {"dims": rot_dims or dim // 2, "base": 500000.0}}
    right = {"heads": memory_heads, "dim": memory_dim, "vdim": memory_vdim, "gate_cap": 15.0}
    return delta, left, right


def _fepopel_preset(pattern: str, loop: tuple[int, int, int], vocab: int, width: int, heads: int,
                    dim: int, rot_dim: int, rank: int, kv_heads: int, chunk: int, ff: int,
                    experts: int, top: int, expert_ff: int, shared_ff: int) -> dict:
    """``pattern``: two letters per layer, l for latent or c for chunked attention, then d for a
    dense feed-forward or e for experts."""
    mixers = {
        "l": ("latent_attention", {
            "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": dim, "kv_rank": rank,
            "scale": (dim + rot_dim) ** -0.5, "rot": {"dims": rot_dim, "base": 500000.0}}),
        "c": ("attention", {
            "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
            "softcap": 50.0, "mask": {"size": chunk}})}
    mlps = {"d": {"kind": "dense", "ff": ff},
            "e": {"kind": "moe", "router": {"experts": experts, "top": top, "scale": 2.0},
                  "expert": {"ff": expert_ff}, "shared": {"ff": shared_ff}}}
    return {"architecture": "Fepopel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
            "embedding": {"scale": width ** 0.5},
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]},
            "layers": [{"type": mixers[p[0]][0], "mixer": mixers[p[0]][1], "mlp": mlps[p[1]]}
                       for p in pattern.split()]}


def _vadelix_preset(pattern: str, vocab: int, width: int, heads: int, kv_heads: int, dim: int,
                    window: int, wkv_heads: int, wkv_dim: int, ff: int, experts: int, top: int,
                    groups: tuple[int, int], expert_ff: int, shared_ff: int, rank: int) -> dict:
    """``pattern``: two letters per layer, r for rotary attention, b for windowed attention with
    distance biases or w for time mixing, then d for a dense feed-forward or e for experts."""
    size = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5,
            "v_mix": True}
    mixers = {
        "r": ("attention", {**size, "rot": {
            "dims": dim // 2, "base": 500000.0,
            "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}),
        "b": ("attention_2", {**size, "mask": {"size": window},
                              "q_temp": {"coef": 0.1, "every": 8192}}),
        "w": ("wkv", {"heads": wkv_heads, "dim": wkv_dim, "decay_rank": rank})}
    mlps = {"d": {"kind": "dense", "ff": ff},
            "e": {"kind": "moe", "expert": {"ff": expert_ff}, "shared": {"ff": shared_ff},
                  "router": {"experts": experts, "top": top,
                             "groups": {"count": groups[0], "keep": groups[1]}}}}
    return {"architecture": "Vadelix", "vocab": vocab, "width": width, "residual_mult": 0.5,
            "norm": {"eps": 1e-5, "groups": 8}, "canon": {"taps": 4},
            "layers": [{"type": mixers[p[0]][0], "mixer": mixers[p[0]][1], "mlp": mlps[p[1]]}
                       for p in pattern.split()]}


#: configurations of designs that are described layer by layer
_LAYER_LIST_PRESETS: dict[str, dict] = {
    "tiny-sapapel": _sapapel_preset(3, 1024, 128, 4, 24, 40, 48, 6, 2, 48),
    # layers of the size of DeepSeek-V2-Lite's
    "sapapel-16b": _sapapel_preset(27, 102400, 2048, 16, 128, 128, 512, 64, 6, 1408),
    "tiny-fepopel": _fepopel_preset("ld le ce le", (1, 3, 2), 1024, 128, 4, 24, 8, 48, 2, 32, 192,
                                    6, 2, 48, 40),
    # layers of the size of DeepSeek-V2-Lite's
    "fepopel-16b": _fepopel_preset("ld" + " le ce le" * 8 + " le", (1, 4, 2), 102400, 2048, 16, 128,
                                   64, 512, 4, 1024, 10944, 64, 6, 1408, 2816),
    "tiny-vadelix": _vadelix_preset("rd we be rd", 1024, 128, 4, 2, 24, 32, 4, 24, 192, 8, 2, (4, 2),
                                    48, 40, 12),
    # layers of the size of Llama-3-8B's, experts of the size of DeepSeek-V2-Lite's
    "vadelix-12b": _vadelix_preset("rd we be we" + " rd we be we" * 7, 128256, 4096, 32, 8, 128,
                                   1024, 64, 64, 14336, 32, 4, (4, 2), 1536, 3072, 64),
    "tiny-fizunex": _fizunex_preset("dpd", 1024, 128, 192, *_fizunex_mixers(4, 2, 32, 2, 24, 40)),
    # layers of the size of Llama-3-8B's
    "fizunex-8b": _fizunex_preset("dddp" * 8, 128256, 4096, 14336,
                                  *_fizunex_mixers(32, 8, 128, 8, 128, 256)),
}


@dataclass
class CacheConfig:
    block_size: int = 16
    gpu_memory_utilization: float = 0.90
    num_gpu_blocks: Optional[int] = None   # override of the profiled value
    num_cpu_blocks: int = 0                # swap space
    enable_prefix_caching: bool = True
    cache_dtype: str = "auto"


@dataclass
class SchedulerConfig:
    max_num_seqs: int = 256
    max_num_batched_tokens: int = 8192
    max_model_len: int = 8192
    enable_chunked_prefill: bool = True
    policy: str = "fcfs"                   # or "priority"
    async_scheduling: bool = False
    num_scheduler_steps: int = 1           # multi-step decode (device-side advance)
    long_prefill_token_threshold: int = 0


@dataclass
class ParallelConfig:
    tensor_parallel_size: int = 1
    pipeline_parallel_size: int = 1
    data_parallel_size: int = 1
    enable_expert_parallel: bool = False
    enable_sequence_parallel: bool = False
    comm_backend: str = "fused"            # "fused" (symmetric-memory kernels) | "nccl"
    num_redundant_experts: int = 0
    enable_eplb: bool = False

    @property
    def world_size(self) -> int:
        return self.tensor_parallel_size * self.pipeline_parallel_size * self.data_parallel_size


@dataclass
class SpeculativeConfig:
    method: Optional[str] = None           # "ngram" | "mtp" | "draft_model"
    num_speculative_tokens: int = 0
    prompt_lookup_max: int = 4
    prompt_lookup_min: int = 1
    draft_model: Optional[str] = None


@dataclass
class EngineConfig:
    model: ModelConfig
    cache: CacheConfig = field(default_factory=CacheConfig)
    scheduler: SchedulerConfig = field(default_factory=SchedulerConfig)
    parallel: ParallelConfig = field(default_factory=ParallelConfig)
    speculative: SpeculativeConfig = field(default_factory=SpeculativeConfig)
    device: str = "auto"
    seed: int = 0
    enforce_eager: bool = False
    cuda_graph_sizes: Optional[list[int]] = None
    load_format: str = "dummy"             # "dummy" (random init) | "safetensors"
    model_path: Optional[str] = None
    quantization_param_path: Optional[str] = None   # JSON with the scales of an 8-bit KV cache
    additional_config: dict = field(default_factory=dict)

    def __post_init__(self) -> None:
        if self.device == "auto":
            self.device = "cuda" if torch.cuda.is_available() else "cpu"
        self.scheduler.max_model_len = min(self.scheduler.max_model_len,
                                           self.model.max_position_embeddings)
        if not self.scheduler.enable_chunked_prefill:
            self.scheduler.max_num_batched_tokens = max(self.scheduler.max_num_batched_tokens,
                                                        self.scheduler.max_model_len)
