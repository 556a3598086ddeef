"""Fizunex: gated delta rule layers beside layers that run attention and a matrix memory in
parallel; norms on the sublayers' outputs only.

    x = x + norm1(mixer(x))
    x = x + norm2(dense(x))          (layers with a feed-forward)

The residual stream, the norms and the recurrent states are fp32; matrix products run in the
model's dtype.  Sizes and constants come from the configuration's layer list
(``ModelConfig.layer_specs``), layer by layer.  Keys and values live in the paged cache, recurrent
states in one slot per running request.
"""
from __future__ import annotations

from typing import Iterable, Optional

import torch
import torch.nn as nn

from .. import ops
from ..config import AttentionSpec, DeltaSpec, LayerSpec, MemorySpec, ModelConfig
from ..layers.attention import AttentionMetadata
from ..layers.basic import LayerNormParams, ParallelLMHead, RotaryEmbedding
from ..layers.key_attention import KeyAttention
from ..layers.mixer import MixerBlock
from ..layers.recurrent import GatedDelta, MatrixMemory
from ..ops import cuda as C
from ..ops import ref
from ..parallel.state import get_state
from .decoder import DecoderLM, DenseMLP


class FizunexLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: LayerSpec, device, prefix: str, rotary):
        super().__init__()
        eps, dt, H = cfg.rms_norm_eps, cfg.dtype, cfg.hidden_size
        parts = []
        for name, scale, s in spec.parts:
            p = f"{prefix}.mix.{name}"
            if isinstance(s, DeltaSpec):
                part = GatedDelta(s, eps, dt, device, p)
            elif isinstance(s, MemorySpec):
                part = MatrixMemory(s, eps, dt, device, p)
            elif isinstance(s, AttentionSpec):
                part = KeyAttention(s, eps, dt, device, p, rotary(s))
            else:
                raise ValueError(f"{p}: unknown mixer {type(s).__name__}")
            parts.append((name, scale, part))
        self.mix = MixerBlock(parts, H, dt, device, prefix + ".mix")
        self.norm1 = LayerNormParams(H, device)
        self.mlp = DenseMLP(cfg, H, spec.intermediate_size, device, prefix + ".mlp") \
            if spec.has_mlp else None
        self.norm2 = LayerNormParams(H, device) if spec.has_mlp else None


class FizunexForCausalLM(DecoderLM):
    # CUDA sources with the kernels of this model (a fresh checkout may build only these)
    native_sources = ("activation", "attention", "attention_any", "attention_fmha",
                      "attention_tma", "cache", "common", "gemm_bf16", "gemm_pair", "gemm_skinny",
                      "recurrent", "residual", "sampler", "step")
    # recurrent states cannot be taken back and are not part of the cache blocks: no draft tokens,
    # no prefix cache, no swapping of blocks
    has_request_state = True

    def __init__(self, cfg: ModelConfig, device="cpu"):
        nn.Module.__init__(self)
        st = get_state()
        if cfg.layer_specs is None:
            raise ValueError("a Fizunex configuration lists its layers")
        if st.pp.world_size > 1 or st.dp.world_size > 1 or st.ep.world_size > 1:
            raise ValueError("Fizunex runs with tensor parallelism only")
        if cfg.quantization:
            raise ValueError("there is no quantised Fizunex checkpoint format")
        if cfg.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"Fizunex runs in bfloat16 or float32, not {cfg.dtype}")
        self.cfg = cfg
        self.device = torch.device(device)
        self.start_layer, self.end_layer = 0, cfg.num_hidden_layers
        self.is_first_stage = self.is_last_stage = True
        if self.device.type == "cuda" and cfg.dtype == torch.float32:
            # 32-bit means 32-bit: no reduced-precision mode of the library's matrix products
            torch.backends.cuda.matmul.allow_tf32 = False
        self.embed_tokens = ParallelLMHead(cfg.vocab_size, cfg.hidden_size, cfg.dtype, device)
        self.lm_head = None                         # the embedding table is the output projection
        tables: dict = {}

        def rotary(s: AttentionSpec) -> RotaryEmbedding:
            key = (s.rot_dims, s.rot_base)
            if key not in tables:                   # one table per kind of rotation
                tables[key] = RotaryEmbedding(s.head_dim, s.rot_dims, cfg.max_position_embeddings,
                                              s.rot_base, is_neox=False, device=device,
                                              keep_fp32=True)
            return tables[key]

        self.layers = nn.ModuleList(FizunexLayer(cfg, s, device, f"l{i}", rotary)
                                    for i, s in enumerate(cfg.layer_specs))
        self.norm = LayerNormParams(cfg.hidden_size, device)

    def kv_cache_spec(self) -> dict:
        shapes = [layer.mix.cache_shape() for layer in self.layers]
        kv = [s for s in shapes if s is not None]
        heads = [p.H for layer in self.layers for p in layer.mix.parts
                 if isinstance(p, KeyAttention)]
        return {"type": "gqa", "layers": len(shapes), "layer_shapes": shapes,
                # the largest layer sizes the shared workspace of split decode attention
                "kv_heads": max((h for h, _ in kv), default=1),
                "head_dim": max((d for _, d in kv), default=1), "q_heads": max(heads, default=1),
                "request_state": [layer.mix.state_shapes() for layer in self.layers]}

    def forward(self, input_ids: Optional[torch.Tensor], md: AttentionMetadata,
                kv_caches: list[torch.Tensor], intermediate=None,
                inputs_embeds: Optional[torch.Tensor] = None):
        cfg = self.cfg
        emb = inputs_embeds if inputs_embeds is not None else self.embed_tokens(input_ids)
        o_ = C if ops.use_native(emb) else ref
        x, lo = o_.start_rows(emb, cfg.embed_scale)
        if emb.shape[0] == 0:
            return lo
        end = dict(final_weight=self.norm.weight, final_bias=self.norm.bias,
                   final_scale=cfg.logit_scale)
        for i, layer in enumerate(self.layers):
            last = i + 1 == len(self.layers)
            state = md.request_state[i] if md.request_state else None
            y = layer.mix(lo, md, kv_caches[i] if kv_caches else None, state)
            lo = torch.empty_like(lo)
            layer.norm1.add(o_, x, y, cfg.rms_norm_eps, lo, end if last and not layer.mlp else {})
            if layer.mlp is not None:
                y = layer.mlp(lo)
                lo = torch.empty_like(lo)
                layer.norm2.add(o_, x, y, cfg.rms_norm_eps, lo, end if last else {})
        return lo

    # -- weights --------------------------------------------------------------------
    _MLP = {"gate": ("gate_up_proj", 0), "up": ("gate_up_proj", 1), "down": ("down_proj", None)}

    def _load_one(self, name: str, t: torch.Tensor) -> bool:
        """False for a tensor that the configuration does not ask for."""
        if name == "embed":
            self.embed_tokens.load_weight("weight", t)
            return True
        if name in ("final.norm", "final.norm.b"):
            self.norm.load_weight("bias" if name.endswith(".b") else "weight", t)
            return True
        head, _, rest = name.partition(".")
        if not (head[:1] == "l" and head[1:].isdigit() and int(head[1:]) < len(self.layers)):
            return False
        layer = self.layers[int(head[1:])]
        part, _, sub = rest.partition(".")
        if part in ("norm1", "norm2") and sub in ("", "b") and getattr(layer, part) is not None:
            getattr(layer, part).load_weight("bias" if sub else "weight", t)
        elif part == "mix":
            return layer.mix.load(sub, t)
        elif part == "mlp" and layer.mlp is not None and sub in self._MLP:
            owner, shard = self._MLP[sub]
            getattr(layer.mlp, owner).load_weight("weight", t, shard)
        else:
            return False
        return True

    def _expected_tensors(self) -> set[str]:
        names = {"embed", "final.norm", "final.norm.b"}
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            names |= {p + "norm1", p + "norm1.b"} | {p + "mix." + n
                                                     for n in layer.mix.tensor_names()}
            if layer.mlp is not None:
                names |= {p + "norm2", p + "norm2.b"} | {p + "mlp." + n for n in self._MLP}
        return names

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]) -> set[str]:
        loaded = {name for name, t in weights if self._load_one(name, t)}
        missing = self._expected_tensors() - loaded
        if missing:
            raise ValueError(f"{len(missing)} tensors are missing from the checkpoint, e.g. "
                             f"{sorted(missing)[:3]}")
        self.finalize_weights()
        return loaded

    @torch.no_grad()
    def init_random(self, seed: int = 0, std: float = 0.02) -> None:
        """Random weights as in the other families; norm weights one, forget gates and decays that
        keep a state for some hundred tokens."""
        super().init_random(seed, std)
        for m in self.modules():
            if isinstance(m, LayerNormParams):
                m.weight.fill_(1.0)
                m.bias.zero_()
            elif isinstance(m, GatedDelta):
                m.norm.fill_(1.0)
                m.a_log.fill_(-1.0)
                m.dt_bias.fill_(-4.0)
            elif isinstance(m, MatrixMemory):
                m.norm.fill_(1.0)
                m.i_bias.zero_()
                m.f_bias.fill_(5.0)
            elif isinstance(m, KeyAttention):
                m.q_norm.fill_(1.0)
                m.k_norm.fill_(1.0)
                m.sink.zero_()
