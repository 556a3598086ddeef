"""Fepopel: latent attention with sinks and head gates beside chunked attention, squared-ReLU experts,
norms before and after every sublayer, and a run of layers that is passed through several times.

    x = x + norm1b(mixer(norm1(x)))
    x = x + norm2b(ff(norm2(x)))          (layers with a feed-forward)

In front of every pass of the loop a vector of that pass is added to x.  A pass has the weights of
the others and a cache of its own, so the model's caches are numbered by layer runs
(``ModelConfig.layer_runs``), not by layers.  Every norm is fused with the residual sum in front of
it: one kernel normalises a sublayer's output (for experts: weights and sums their rows first), adds
it and the vector of the next pass to the fp32 stream, and normalises the new row for the next
sublayer.  The residual stream and the norms are fp32; matrix products run in the model's dtype.
Sizes and constants come from the configuration's layer list (``ModelConfig.layer_specs``).
"""
from __future__ import annotations

from typing import Iterable, Optional

import torch
import torch.nn as nn

from .. import ops
from ..config import LayerSpec, ModelConfig
from ..layers.attention import AttentionMetadata
from ..layers.basic import (ParallelLMHead, RMSNormParams, VocabParallelEmbedding,
                            build_cos_sin_cache)
from ..layers.key_attention import ChunkAttention
from ..layers.latent import LatentAttention
from ..layers.mixer import MixerBlock
from ..layers.moe import GatedSharedMoE
from ..ops import cuda as C
from ..ops import ref
from ..parallel.state import get_state
from .decoder import DecoderLM, DenseMLP


class FepopelLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: LayerSpec, device, prefix: str, table):
        super().__init__()
        eps, dt, H = cfg.rms_norm_eps, cfg.dtype, cfg.hidden_size
        if spec.parts:
            self.mix = MixerBlock([(n, f, ChunkAttention(s, eps, dt, device, prefix + ".mix"))
                                   for n, f, s in spec.parts], H, dt, device, prefix + ".mix")
        else:
            self.mix = LatentAttention(spec, H, eps, dt, device, prefix + ".mix", table(spec))
        self.norm1, self.norm1b = RMSNormParams(H, device), RMSNormParams(H, device)
        self.mlp = None
        if spec.num_experts:
            self.mlp = GatedSharedMoE(spec.num_experts, spec.num_experts_per_tok,
                                      spec.router_scale, H, spec.moe_intermediate_size,
                                      spec.shared_intermediate_size, dt, device, prefix + ".mlp")
        elif spec.intermediate_size:
            self.mlp = DenseMLP(cfg, H, spec.intermediate_size, device, prefix + ".mlp")
        if self.mlp is not None:
            self.norm2, self.norm2b = RMSNormParams(H, device), RMSNormParams(H, device)

    def attend(self, h: torch.Tensor, md: AttentionMetadata, cache: Optional[torch.Tensor]
               ) -> torch.Tensor:
        if isinstance(self.mix, MixerBlock):
            return self.mix(h, md, cache, None)
        return self.mix(h, cache, md)

    def feed_forward(self, h: torch.Tensor) -> tuple[torch.Tensor, dict]:
        return self.mlp(h) if isinstance(self.mlp, GatedSharedMoE) else (self.mlp(h), {})

    def norms(self) -> list[str]:
        return ["norm1", "norm1b"] + (["norm2", "norm2b"] if self.mlp is not None else [])

    _DENSE = {"gate": ("gate_up_proj", 0), "up": ("gate_up_proj", 1), "down": ("down_proj", None)}

    def load(self, name: str, t: torch.Tensor) -> bool:
        """False if the layer has no tensor of that name."""
        part, _, sub = name.partition(".")
        if name in self.norms():
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
        return set(self.norms()) | {"mix." + n for n in self.mix.tensor_names()} | {
            "mlp." + n for n in mlp}


class FepopelForCausalLM(DecoderLM):
    # CUDA sources with the kernels of this model (a fresh checkout may build only these)
    native_sources = ("activation", "attention", "attention_any", "attention_fmha",
                      "attention_mla", "attention_tma", "cache", "common", "gemm_bf16",
                      "gemm_pair", "gemm_skinny", "latent", "moe", "residual", "sampler", "step")

    def __init__(self, cfg: ModelConfig, device="cpu"):
        nn.Module.__init__(self)
        st = get_state()
        if cfg.layer_specs is None:
            raise ValueError("a Fepopel configuration lists its layers")
        if st.pp.world_size > 1 or st.dp.world_size > 1 or st.ep.world_size > 1:
            raise ValueError("Fepopel runs with tensor parallelism only")
        if cfg.quantization:
            raise ValueError("there is no quantised Fepopel checkpoint format")
        if cfg.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"Fepopel runs in bfloat16 or float32, not {cfg.dtype}")
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

        def table(s: LayerSpec) -> torch.Tensor:
            key = (s.rot_dim, s.rot_base)
            if key not in tables:                   # one table per kind of rotation
                tables[key] = build_cos_sin_cache(*key[:1], cfg.max_position_embeddings, key[1],
                                                  dtype=torch.float64).float().to(device)
            return tables[key]

        self.layers = nn.ModuleList(FepopelLayer(cfg, s, device, f"l{i}", table)
                                    for i, s in enumerate(cfg.layer_specs))
        self.runs = cfg.layer_runs
        self.loop_step = nn.Parameter(torch.zeros(cfg.loop[2], H, dtype=torch.float32,
                                                  device=device), requires_grad=False) \
            if cfg.loop else None
        self.norm = RMSNormParams(H, device)
        self.lm_head = ParallelLMHead(cfg.vocab_size, H, cfg.dtype, device)

    @property
    def num_local_layers(self) -> int:
        """Caches of the model: one per layer run."""
        return len(self.runs)

    def kv_cache_spec(self) -> dict:
        mixes = [self.layers[i].mix for i, _ in self.runs]
        shapes = [m.cache_shape() if isinstance(m, MixerBlock) else (m.W,) for m in mixes]
        kv = [s for s in shapes if len(s) == 2]
        heads = [p.H for m in mixes if isinstance(m, MixerBlock) for p in m.parts]
        return {"type": "layers", "layers": len(shapes), "layer_shapes": shapes,
                # the largest layer sizes the shared workspace of split decode attention
                "kv_heads": max((h for h, _ in kv), default=1),
                "head_dim": max((d for _, d in kv), default=1), "q_heads": max(heads, default=1)}

    def forward(self, input_ids: Optional[torch.Tensor], md: AttentionMetadata,
                kv_caches: list[torch.Tensor], intermediate=None,
                inputs_embeds: Optional[torch.Tensor] = None):
        cfg, eps = self.cfg, self.cfg.rms_norm_eps
        emb = inputs_embeds if inputs_embeds is not None else self.embed_tokens(input_ids)
        o_ = C if ops.use_native(emb) else ref

        def entry(r: int) -> dict:
            """What the kernel in front of layer run r adds to the stream and normalises it with."""
            if r == len(self.runs):
                return dict(step=None, weight=self.norm.weight)
            i, t = self.runs[r]
            return dict(step=None if t is None else self.loop_step[t],
                        weight=self.layers[i].norm1.weight)

        x, lo = o_.start_rows(emb, cfg.embed_scale, eps=eps, **entry(0))
        if emb.shape[0] == 0:
            return lo

        def add(y: torch.Tensor, norm: RMSNormParams, step, weight, last: bool, rows: dict
                ) -> torch.Tensor:
            out = torch.empty_like(lo)
            o_.add_normed(x, y, norm.weight, None, eps, out, out=None if last else x,
                          layer_norm=False, final_weight=weight, step=step, **rows)
            return out

        for r, (i, _) in enumerate(self.runs):
            layer, nxt, last = self.layers[i], entry(r + 1), r + 1 == len(self.runs)
            y = layer.attend(lo, md, kv_caches[r] if kv_caches else None)
            if layer.mlp is not None:
                lo = add(y, layer.norm1b, None, layer.norm2.weight, False, {})
                y, rows = layer.feed_forward(lo)
                lo = add(y, layer.norm2b, last=last, rows=rows, **nxt)
            else:
                lo = add(y, layer.norm1b, last=last, rows={}, **nxt)
        return lo

    # -- weights --------------------------------------------------------------------
    _TOP = {"embed": "embed_tokens", "head": "lm_head", "final.norm": "norm"}

    def _load_one(self, name: str, t: torch.Tensor) -> bool:
        """False for a tensor that the configuration does not ask for."""
        if name in self._TOP:
            getattr(self, self._TOP[name]).load_weight("weight", t)
            return True
        if name == "loop.step" and self.loop_step is not None:
            self.loop_step.data.copy_(t)
            return True
        head, _, rest = name.partition(".")
        if not (head[:1] == "l" and head[1:].isdigit() and int(head[1:]) < len(self.layers)):
            return False
        return self.layers[int(head[1:])].load(rest, t)

    def _expected_tensors(self) -> set[str]:
        names = set(self._TOP) | ({"loop.step"} if self.loop_step is not None else set())
        return names | {f"l{i}.{n}" for i, layer in enumerate(self.layers)
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
        """Random weights as in the other families; norm weights one, sinks zero."""
        super().init_random(seed, std)
        for m in self.modules():
            if isinstance(m, RMSNormParams):
                m.weight.fill_(1.0)
            elif isinstance(m, LatentAttention):
                m.latent_norm.fill_(1.0)
                m.sink.zero_()
            elif isinstance(m, ChunkAttention):
                m.q_norm.fill_(1.0)
                m.k_norm.fill_(1.0)
