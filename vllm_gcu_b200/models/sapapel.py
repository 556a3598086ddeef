"""Sapapel: latent attention without positions behind a token shift, input-weighted experts,
norms after the residual sums, and a depth-weighted average of all results after every layer.

With X_0 the embedding output and alpha from the configuration, layer i computes

    h       = x + (x_prev - x) * mu                       (token shift, h feeds the mixer)
    x'      = rms(alpha x + mixer(h)) * g1
    X_(i+1) = rms(alpha x' + experts(x')) * g2            (x' itself without a feed-forward)
    x       = sum_j w_j X_j,  j = 0 .. i+1

The residual stream, the norms, the router scores, the averages and the shift's state are fp32;
matrix products run in the model's dtype.  Sizes and constants come from the configuration's
layer list (``ModelConfig.layer_specs``), layer by layer.
"""
from __future__ import annotations

import dataclasses
from typing import Iterable, Optional

import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import ops
from ..config import LayerSpec, ModelConfig
from ..layers.attention import AttentionMetadata
from ..layers.basic import ParallelLMHead, ScalarGain, VocabParallelEmbedding
from ..layers.latent import LatentAttention, TokenShift
from ..layers.linear import ReplicatedLinear
from ..layers.moe import InputWeightedMoE, select_experts
from ..ops import cuda as C
from ..ops import ref
from ..parallel.communicator import get_comm
from ..parallel.state import get_state, tp_size
from .decoder import DecoderLM


class RoutedExperts(nn.Module):
    """fp32 sigmoid router + experts with weighted inputs.  Returns what ``post_norm`` takes."""

    def __init__(self, cfg: ModelConfig, spec: LayerSpec, device, prefix: str):
        super().__init__()
        self.k = spec.num_experts_per_tok
        self.route_cfg = dataclasses.replace(
            cfg, num_experts=spec.num_experts, num_experts_per_tok=self.k, n_group=1,
            topk_group=1, routed_scaling_factor=1.0, scoring_func="sigmoid", norm_topk_prob=False)
        self.router = ReplicatedLinear(cfg.hidden_size, spec.num_experts, dtype=cfg.dtype,
                                       device=device, prefix=prefix + ".router")
        self.experts = InputWeightedMoE(spec.num_experts, cfg.hidden_size,
                                        spec.moe_intermediate_size, cfg.dtype, device,
                                        prefix + ".experts")

    def forward(self, x: torch.Tensor, x_lo: torch.Tensor):
        """``x [T, H]`` fp32, ``x_lo`` the same rows in the model's dtype."""
        w = self.router.weight
        if ops.use_native(x) and x_lo.dtype == torch.bfloat16:
            z = C.gemm_bf16(x_lo, w, epilogue=C.EPI_FP32)
        else:
            z = F.linear(x_lo.float(), w.float())
        topk_w, topk_ids = select_experts(z, self.route_cfg)
        y, pos_of = self.experts(x, topk_w, topk_ids)
        if tp_size() == 1:
            return y, pos_of
        # every rank has its slice of the intermediate dimension: sum slots, then ranks
        T, H = x.shape
        p = pos_of.view(-1)[:T * self.k].view(T, self.k).long()
        dense = y[p.clamp(min=0)].float().mul_((p >= 0).unsqueeze(-1)).sum(1)[:, :H]
        return get_comm("tp").all_reduce(dense.to(x_lo.dtype).contiguous()), None


class SapapelLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, idx: int, device):
        super().__init__()
        spec = cfg.layer_specs[idx]
        p = f"l{idx}"
        self.idx, self.alpha, self.eps = idx, cfg.residual_alpha, cfg.rms_norm_eps
        self.shift = TokenShift(cfg.hidden_size, device)
        self.mix = LatentAttention(spec, cfg.hidden_size, cfg.rms_norm_eps, cfg.dtype, device,
                                   p + ".mix")
        self.norm1 = ScalarGain(device)
        self.mlp = RoutedExperts(cfg, spec, device, p + ".mlp") if spec.has_mlp else None
        self.norm2 = ScalarGain(device) if spec.has_mlp else None
        self.dwa = nn.Parameter(torch.zeros(idx + 2, dtype=torch.float32, device=device),
                                requires_grad=False)


class SapapelForCausalLM(DecoderLM):
    # CUDA sources with the kernels of this model (a fresh checkout may build only these)
    native_sources = ("common", "attention_mla", "gemm_bf16", "gemm_pair", "gemm_skinny", "latent",
                      "moe", "residual", "sampler", "step", "cache")
    # the shift's state follows the cache blocks; a rejected draft token would leave its row there
    has_block_state = True

    def __init__(self, cfg: ModelConfig, device="cpu"):
        nn.Module.__init__(self)
        st = get_state()
        if cfg.layer_specs is None:
            raise ValueError("a Sapapel configuration lists its layers")
        if st.pp.world_size > 1 or st.dp.world_size > 1 or st.ep.world_size > 1:
            raise ValueError("Sapapel runs with tensor parallelism only: the depth average reads "
                             "the results of all layers, the experts are sharded within a replica")
        if cfg.quantization:
            raise ValueError("there is no quantised Sapapel checkpoint format")
        if cfg.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"Sapapel runs in bfloat16 or float32, not {cfg.dtype}")
        self.cfg = cfg
        self.device = torch.device(device)
        self.start_layer, self.end_layer = 0, cfg.num_hidden_layers
        self.is_first_stage = self.is_last_stage = True
        if self.device.type == "cuda" and cfg.dtype == torch.float32:
            # 32-bit means 32-bit: no reduced-precision mode of the library's matrix products
            torch.backends.cuda.matmul.allow_tf32 = False
        self.embed_tokens = VocabParallelEmbedding(cfg.vocab_size, cfg.hidden_size, cfg.dtype,
                                                   device)
        self.layers = nn.ModuleList(SapapelLayer(cfg, i, device)
                                    for i in range(cfg.num_hidden_layers))
        self.norm = ScalarGain(device)
        self.lm_head = ParallelLMHead(cfg.vocab_size, cfg.hidden_size, cfg.dtype, device)

    def kv_cache_spec(self) -> dict:
        H = self.cfg.hidden_size
        return {"type": "mla", "layers": len(self.layers),
                "widths": [layer.mix.W for layer in self.layers],
                "block_state": [H] * len(self.layers)}

    def forward(self, input_ids: Optional[torch.Tensor], md: AttentionMetadata,
                kv_caches: list[torch.Tensor], intermediate=None,
                inputs_embeds: Optional[torch.Tensor] = None):
        cfg, n = self.cfg, len(self.layers)
        emb = inputs_embeds if inputs_embeds is not None else self.embed_tokens(input_ids)
        T, H, dt = emb.shape[0], cfg.hidden_size, cfg.dtype
        dev = emb.device
        new = lambda *s: torch.empty(*s, dtype=torch.float32, device=dev)  # noqa: E731
        hist = new(n, T, H)                   # X_0 .. X_(n-1); X_n is used at once
        hist[0].copy_(emb)
        if T == 0:
            return torch.empty(0, H, dtype=dt, device=dev)
        x, avg, mid = hist[0], new(T, H), new(T, H)
        mid_lo = torch.empty(T, H, dtype=dt, device=dev)
        hidden = torch.empty(T, H, dtype=dt, device=dev)
        post_norm = C.post_norm if ops.use_native(emb) else ref.post_norm
        for i, layer in enumerate(self.layers):
            cache = kv_caches[i] if kv_caches else None
            state = md.block_state[i] if md.block_state and not md.is_dummy else None
            bs = cache.shape[1] if cache is not None else 1
            h = layer.shift(x, dt, md, state, bs)
            y = layer.mix(h, cache, md, x, state)
            last = i + 1 == n
            tail = dict(res=None if last else hist[i + 1], hist=hist, n=i + 1, weights=layer.dwa,
                        avg=None if last else avg,
                        final_gain=self.norm.gain if last else None, lo=hidden if last else None)
            if layer.mlp is None:
                post_norm(x, y, layer.norm1.gain, layer.alpha, layer.eps, **tail)
            else:
                post_norm(x, y, layer.norm1.gain, layer.alpha, layer.eps, res=mid, lo=mid_lo)
                y, pos_of = layer.mlp(mid, mid_lo)
                post_norm(mid, y, layer.norm2.gain, layer.alpha, layer.eps, pos_of=pos_of,
                          k=layer.mlp.k, **tail)
            x = avg
        return hidden

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
        layer = self.layers[int(head[1:])]
        part, _, sub = rest.partition(".")
        if rest == "dwa":
            layer.dwa.data.copy_(t)
        elif rest == "shift":
            layer.shift.load_weight("weight", t)
        elif rest == "norm1":
            layer.norm1.load_weight("weight", t)
        elif part == "mix":
            layer.mix.load_weight(sub, t)
        elif layer.mlp is None:
            return False
        elif rest == "norm2":
            layer.norm2.load_weight("weight", t)
        elif rest == "mlp.router":
            layer.mlp.router.load_weight("weight", t)
        elif part == "mlp" and sub[:1] == "e":
            e, _, which = sub[1:].partition(".")
            layer.mlp.experts.load_expert_weight(int(e), which, t)
        else:
            return False
        return True

    def _expected_tensors(self) -> set[str]:
        names = set(self._TOP)
        for i, s in enumerate(self.cfg.layer_specs):
            p = f"l{i}."
            names |= {p + k for k in ("norm1", "shift", "dwa")}
            names |= {p + "mix." + k for k in ("q", "dkv", "dkv.norm", "uk", "uv", "g", "o")}
            if s.has_mlp:
                names |= {p + "norm2", p + "mlp.router"}
                names |= {f"{p}mlp.e{e}.{k}" for e in range(s.num_experts)
                          for k in ("gate", "up", "down")}
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
        """Random weights as in the other families; gains one, shift fractions a half, and an
        average that passes on the newest result with a little of all earlier ones."""
        super().init_random(seed, std)
        for layer in self.layers:
            layer.shift.mu.fill_(0.5)
            layer.mix.latent_norm.fill_(1.0)
            layer.dwa.fill_(0.1 / max(1, layer.idx + 1))
            layer.dwa[-1] = 1.0
            for g in (layer.norm1, layer.norm2):
                if g is not None:
                    g.gain.fill_(1.0)
        self.norm.gain.fill_(1.0)
