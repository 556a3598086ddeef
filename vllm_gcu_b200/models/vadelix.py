"""Vadelix: attention layers of two kinds beside linear recurrences, a causal convolution in front of
every mixer, values mixed with those of the first layer, grouped norms in front of the sublayers.

    x = x + m * mixer(conv(norm1(x)))
    x = x + m * ff(norm2(x))          (layers with a feed-forward)

Rotary attention normalises its whole query and key projections and every head's values and has a
learnt sink per head; windowed attention has no rotation but distance biases, a temperature of its
queries by position and a zero sink; time mixing keeps a matrix per head.  Feed-forwards are dense
(GELU-gated), or routed GELU experts of the best groups beside a shared one.

The residual stream, the norms and the recurrent states are fp32; matrix products run in the model's
dtype.  One kernel between two sublayers adds the result (for experts: weights and sums their rows
first), normalises the new row and, for single tokens, convolves and mixes it.  Sizes and constants
come from the configuration's layer list (``ModelConfig.layer_specs``), layer by layer.  Keys and values
live in the paged cache, recurrent states and the convolutions' last inputs in one slot per running
request.
"""
from __future__ import annotations

from typing import Iterable, Optional

import torch
import torch.nn as nn

from .. import ops
from ..config import AttentionSpec, LayerSpec, ModelConfig, TimeMixSpec
from ..layers.attention import AttentionMetadata
from ..layers.basic import ParallelLMHead, RMSNormParams, VocabParallelEmbedding
from ..layers.input_conv import InputConv
from ..layers.key_attention import GroupedAttention, rotary_table
from ..layers.mixer import MixerBlock
from ..layers.moe import GatedSharedMoE
from ..layers.recurrent import TimeMix
from ..ops import cuda as C
from ..ops import ref
from ..parallel.state import get_state
from .decoder import DecoderLM, DenseMLP


class VadelixLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: LayerSpec, device, prefix: str, table,
                 first: Optional[AttentionSpec]):
        super().__init__()
        eps, dt, H = cfg.rms_norm_eps, cfg.dtype, cfg.hidden_size
        (_, _, m), = spec.parts
        if isinstance(m, TimeMixSpec):
            self.mix = TimeMix(m, H, eps, dt, device, prefix + ".mix")
        else:
            part = GroupedAttention(m, eps, dt, device, prefix + ".mix", table(m),
                                    first if m.v_mix else None)
            self.mix = MixerBlock([("", 1.0, part)], H, dt, device, prefix + ".mix")
        self.norm1 = RMSNormParams(H, device)
        self.conv = InputConv(H, cfg.conv_taps, dt, device, prefix + ".canon1",
                              getattr(self.mix, "mu", None))
        self.mlp = None
        if spec.num_experts:
            self.mlp = GatedSharedMoE(spec.num_experts, spec.num_experts_per_tok, 1.0, H,
                                      spec.moe_intermediate_size, spec.shared_intermediate_size,
                                      dt, device, prefix + ".mlp", act="gelu",
                                      groups=(spec.router_groups, spec.router_keep),
                                      shared_gate=False)
        elif spec.intermediate_size:
            self.mlp = DenseMLP(cfg, H, spec.intermediate_size, device, prefix + ".mlp",
                                fused_act="gelu_tanh")
        self.norm2 = RMSNormParams(H, device) if self.mlp is not None else None

    def state_shapes(self) -> dict:
        return {**self.conv.state_shapes(),
                **(self.mix.state_shapes() if isinstance(self.mix, TimeMix) else {})}

    def mixer(self, h: torch.Tensor, md: AttentionMetadata, cache: Optional[torch.Tensor],
              state: Optional[dict]) -> torch.Tensor:
        if isinstance(self.mix, TimeMix):
            return self.mix(h, md, state)
        return self.mix(h, md, cache, None)

    def feed_forward(self, h: torch.Tensor) -> tuple[torch.Tensor, dict]:
        return self.mlp(h) if isinstance(self.mlp, GatedSharedMoE) else (self.mlp(h), {})

    _DENSE = {"gate": ("gate_up_proj", 0), "up": ("gate_up_proj", 1), "down": ("down_proj", None)}

    def load(self, name: str, t: torch.Tensor) -> bool:
        """False if the layer has no tensor of that name."""
        part, _, sub = name.partition(".")
        if name == "canon1":
            self.conv.load_weight("weight", t)
            return True
        if name in ("norm1", "norm2") and getattr(self, name) is not None:
            getattr(self, name).load_weight("weight", t)
            return True
        if part == "mix":
            return self.mix.load(sub, t)
        if part != "mlp" or self.mlp is None:
            return False
        if isinstance(self.mlp, GatedSharedMoE):
            return self.mlp.load(sub, t)
        if sub not in self._DENSE:
            return False
        owner, shard = self._DENSE[sub]
        getattr(self.mlp, owner).load_weight("weight", t, shard)
        return True

    def tensor_names(self) -> set[str]:
        mlp = set() if self.mlp is None else self.mlp.tensor_names() \
            if isinstance(self.mlp, GatedSharedMoE) else set(self._DENSE)
        return {"norm1", "canon1"} | ({"norm2"} if self.mlp is not None else set()) | {
            "mix." + n for n in self.mix.tensor_names()} | {"mlp." + n for n in mlp}


class VadelixForCausalLM(DecoderLM):
    # CUDA sources with the kernels of this model (a fresh checkout may build only these)
    native_sources = ("activation", "attention", "attention_any", "attention_fmha",
                      "attention_tma", "cache", "common", "gemm_bf16", "gemm_pair", "gemm_skinny",
                      "group_norm", "moe", "recurrent", "residual", "sampler", "step")
    # recurrent states cannot be taken back and are not part of the cache blocks: no draft tokens,
    # no prefix cache, no swapping of blocks
    has_request_state = True

    def __init__(self, cfg: ModelConfig, device="cpu"):
        nn.Module.__init__(self)
        st = get_state()
        if cfg.layer_specs is None:
            raise ValueError("a Vadelix configuration lists its layers")
        if st.pp.world_size > 1 or st.dp.world_size > 1 or st.ep.world_size > 1:
            raise ValueError("Vadelix runs with tensor parallelism only")
        if cfg.quantization:
            raise ValueError("there is no quantised Vadelix checkpoint format")
        if cfg.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"Vadelix runs in bfloat16 or float32, not {cfg.dtype}")
        self.cfg = cfg
        self.device = torch.device(device)
        self.start_layer, self.end_layer = 0, cfg.num_hidden_layers
        self.is_first_stage = self.is_last_stage = True
        if self.device.type == "cuda" and cfg.dtype == torch.float32:
            # 32-bit means 32-bit: no reduced-precision mode of the library's matrix products
            torch.backends.cuda.matmul.allow_tf32 = False
        H = cfg.hidden_size
        self.embed_tokens = VocabParallelEmbedding(cfg.vocab_size, H, cfg.dtype, device)
        tables: dict = {}

        def table(s: AttentionSpec) -> Optional[torch.Tensor]:
            key = (s.rot_dims, s.rot_base, s.rot_scaling)
            if key not in tables:                   # one table per kind of rotation
                tables[key] = rotary_table(s, cfg.max_position_embeddings, device)
            return tables[key]

        # the layer whose values the later ones mix into theirs
        mixing = [i for i, s in enumerate(cfg.layer_specs)
                  if isinstance(s.parts[0][2], AttentionSpec) and s.parts[0][2].v_mix]
        self.first_mixing = mixing[0] if mixing else -1
        first = cfg.layer_specs[mixing[0]].parts[0][2] if mixing else None
        self.layers = nn.ModuleList(
            VadelixLayer(cfg, s, device, f"l{i}", table, first if i > self.first_mixing else None)
            for i, s in enumerate(cfg.layer_specs))
        self.norm = RMSNormParams(H, device)
        self.lm_head = ParallelLMHead(cfg.vocab_size, H, cfg.dtype, device)

    def kv_cache_spec(self) -> dict:
        shapes = [layer.mix.cache_shape() for layer in self.layers]
        kv = [s for s in shapes if s is not None]
        heads = [p.H for layer in self.layers if isinstance(layer.mix, MixerBlock)
                 for p in layer.mix.parts]
        return {"type": "layers", "layers": len(shapes), "layer_shapes": shapes,
                # the largest layer sizes the shared workspace of split decode attention
                "kv_heads": max((h for h, _ in kv), default=1),
                "head_dim": max((d for _, d in kv), default=1), "q_heads": max(heads, default=1),
                "request_state": [layer.state_shapes() for layer in self.layers]}

    def forward(self, input_ids: Optional[torch.Tensor], md: AttentionMetadata,
                kv_caches: list[torch.Tensor], intermediate=None,
                inputs_embeds: Optional[torch.Tensor] = None):
        cfg, eps = self.cfg, self.cfg.rms_norm_eps
        emb = inputs_embeds if inputs_embeds is not None else self.embed_tokens(input_ids)
        if emb.shape[0] == 0:
            return emb
        o_ = C if ops.use_native(emb) else ref
        x = torch.empty(emb.shape, dtype=torch.float32, device=emb.device)
        if kv_caches and self.first_mixing >= 0 and kv_caches[self.first_mixing] is not None:
            md.first_values = kv_caches[self.first_mixing][1]
        src, y, rows = emb, None, {}          # what the next norm adds up

        def norm(weight: torch.Tensor, last: bool = False):
            def run(lo: torch.Tensor, conv=None) -> torch.Tensor:
                o_.add_group_norm(src, y, cfg.residual_mult, weight, cfg.norm_groups, eps, lo,
                                  out=None if last else x, conv=conv, **rows)
                return lo
            return run

        for i, layer in enumerate(self.layers):
            state = md.request_state[i] if md.request_state else None
            h = layer.conv.after_norm(norm(layer.norm1.weight), emb, md, state)
            y, rows = layer.mixer(h, md, kv_caches[i] if kv_caches else None, state), {}
            src = x
            if layer.mlp is not None:
                h = norm(layer.norm2.weight)(torch.empty_like(emb))
                y, rows = layer.feed_forward(h)
        return norm(self.norm.weight, last=True)(torch.empty_like(emb))

    # -- weights --------------------------------------------------------------------
    _TOP = {"embed": "embed_tokens", "head": "lm_head", "final.norm": "norm"}

    def _load_one(self, name: str, t: torch.Tensor) -> bool:
        """False for a tensor that the configuration does not ask for."""
        if name in self._TOP:
            getattr(self, self._TOP[name]).load_weight("weight", t)
            return True
        head, _, rest = name.partition(".")
        if not (head[:1] == "l" and head[1:].isdigit() and int(head[1:]) < len(self.layers)):
            return False
        return self.layers[int(head[1:])].load(rest, t)

    def _expected_tensors(self) -> set[str]:
        return set(self._TOP) | {f"l{i}.{n}" for i, layer in enumerate(self.layers)
                                 for n in layer.tensor_names()}

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
        """Random weights as in the other families; norm weights one, sinks zero, halves mixed, and
        decays that keep a state for some hundred tokens."""
        super().init_random(seed, std)
        for m in self.modules():
            if isinstance(m, RMSNormParams):
                m.weight.fill_(1.0)
            elif isinstance(m, TimeMix):
                m.mu.fill_(0.5)
                m.w0.fill_(-5.0)
                m.norm.fill_(1.0)
            elif isinstance(m, GroupedAttention):
                for n in ("q_norm", "k_norm"):
                    if getattr(m, n) is not None:
                        getattr(m, n).fill_(1.0)
                if m.spec.sink == "learnt":
                    m.sink.zero_()
                if m.spec.v_mix:
                    m.share.fill_(0.5)
