"""Latent attention without positions, and the token shift in front of it.

``LatentAttention`` caches one normalised latent row per token.  Keys and values of every head
are linear in that row, so they are absorbed: the query is carried into latent space with W_uk,
attention runs over the cached rows themselves (all heads share them), and W_uv expands the
result.  Queries, output gate and latent come from one GEMM.  Steps on the GPU:

1. ``in_proj``: ``[q | gate | latent]`` of the step's rows;
2. one kernel normalises the latent into the paged cache (rows padded with zeros to the tile
   width of the attention kernel) and keeps the rows that a token shift needs later;
3. ``q W_uk``, attention (tcgen05 kernel where the layout allows, csrc/attention_mla.cu, else
   csrc/latent.cu), ``o W_uv``;
4. output gate, ``o_proj``.

``TokenShift`` mixes every row with the row of the token before it.  What it needs of earlier
steps is one fp32 row per request, kept with the request's cache blocks: a block's state row is
the row of the last token written into the block.  A portion that starts at position p reads the
state of the block that holds p - 1, so blocks found by the prefix cache bring their state along,
and freed blocks need no clearing (nothing is read in front of position 0).
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from .. import ops
from ..config import LayerSpec
from ..ops import cuda as C
from ..ops import ref
from ..parallel.state import tp_rank, tp_size
from .attention import AttentionMetadata
from .linear import MixedParallelLinear, RowParallelLinear


def latent_row_width(kv_rank: int, dtype: torch.dtype) -> int:
    """Columns of a cached latent row: whole 64-column tiles where the tcgen05 kernel takes the
    layout, else a multiple of four."""
    if dtype == torch.bfloat16 and kv_rank <= 512:
        return -(-kv_rank // 64) * 64
    return -(-kv_rank // 4) * 4


class TokenShift(nn.Module):
    def __init__(self, hidden: int, device):
        super().__init__()
        self.mu = nn.Parameter(torch.zeros(hidden, dtype=torch.float32, device=device),
                               requires_grad=False)

    def forward(self, x: torch.Tensor, dtype: torch.dtype, md: AttentionMetadata,
                state: Optional[torch.Tensor], block_size: int) -> torch.Tensor:
        op = C.token_shift if ops.use_native(x) else ref.token_shift
        return op(x, self.mu, dtype, state, md.block_tables, md.positions, md.num_decode_tokens,
                  md.cu_q_prefill, block_size)

    def load_weight(self, name: str, full: torch.Tensor, shard_id=None) -> None:
        self.mu.data.copy_(full)


class LatentAttention(nn.Module):
    def __init__(self, spec: LayerSpec, hidden: int, eps: float, dtype, device, prefix: str):
        super().__init__()
        tp = tp_size()
        if spec.num_heads % tp:
            raise ValueError(f"{prefix}: {spec.num_heads} heads over {tp} ranks")
        self.N, self.dim, self.vdim = spec.num_heads // tp, spec.head_dim, spec.v_head_dim
        self.L, self.scale, self.eps = spec.kv_lora_rank, spec.scale, eps
        self.W = latent_row_width(self.L, dtype)
        A = spec.num_heads
        self.in_proj = MixedParallelLinear(hidden, [A * self.dim, A * self.vdim, self.L],
                                           [True, True, False], dtype=dtype, device=device,
                                           prefix=prefix + ".in_proj")
        new = lambda *s: nn.Parameter(torch.zeros(*s, dtype=dtype, device=device),  # noqa: E731
                                      requires_grad=False)
        self.latent_norm = new(self.L)
        self.w_uk = new(self.N, self.dim, self.W)       # columns behind L stay zero
        self.w_uv = new(self.N, self.W, self.vdim)      # rows behind L stay zero
        self.o_proj = RowParallelLinear(A * self.vdim, hidden, dtype=dtype, device=device,
                                        prefix=prefix + ".o_proj")

    _IN = {"q": 0, "g": 1, "dkv": 2}

    def load_weight(self, name: str, full: torch.Tensor, shard_id=None) -> None:
        r, N, L = tp_rank(), self.N, self.L
        if name in self._IN:
            self.in_proj.load_weight("weight", full, self._IN[name])
        elif name == "o":
            self.o_proj.load_weight("weight", full)
        elif name == "dkv.norm":
            self.latent_norm.data.copy_(full)
        elif name == "uk":
            self.w_uk.data[:, :, :L].copy_(full.view(-1, self.dim, L)[r * N:(r + 1) * N])
        elif name == "uv":
            self.w_uv.data[:, :L].copy_(full.view(-1, self.vdim, L)[r * N:(r + 1) * N]
                                        .transpose(1, 2))
        else:
            raise KeyError(name)

    def finalize(self) -> None:
        self.w_uk.data[:, :, self.L:] = 0
        self.w_uv.data[:, self.L:] = 0

    def _attend(self, q: torch.Tensor, cache: torch.Tensor, md: AttentionMetadata) -> torch.Tensor:
        """Causal attention of latent queries ``[T, N, W]`` over the cached rows."""
        T, nd = q.shape[0], md.num_decode_tokens
        if not ops.use_native(q):
            ql = [1] * md.num_decodes + list(md.q_lens_cpu[md.num_decodes:])
            return ref.latent_attention(q, cache, md.block_tables, ql, md.seq_lens_cpu, self.scale,
                                        self.W)
        if not C.mla_attention_supported(q, cache, self.W):
            return C.latent_attention(q, cache, md.block_tables, md.seq_lens, nd, md.cu_q_prefill,
                                      self.scale)
        out = torch.empty_like(q)
        max_len = max(md.max_seq_len, 1)
        if nd > 0:
            C.mla_attention(q[:nd], cache, md.block_tables[:nd], md.seq_lens[:nd], None, nd,
                            max_len, self.scale, out=out[:nd], L=self.W)
        if md.num_prefills > 0:
            B = md.num_decodes + md.num_prefills
            tq = 128 // self.N
            ql = md.q_lens_cpu[md.num_decodes:B]
            n = sum(ql)
            C.mla_attention(q[nd:nd + n], cache, md.block_tables[md.num_decodes:B],
                            md.seq_lens[md.num_decodes:B], md.cu_q_prefill,
                            sum(-(-x // tq) for x in ql), max_len, self.scale,
                            out=out[nd:nd + n], L=self.W)
            nd += n
        if nd < T:
            out[nd:] = 0
        return out

    def forward(self, h: torch.Tensor, kv_cache: Optional[torch.Tensor], md: AttentionMetadata,
                x: Optional[torch.Tensor] = None, state: Optional[torch.Tensor] = None
                ) -> torch.Tensor:
        """``h [T, H]`` projection input.  ``x`` / ``state``: the fp32 rows before the token shift
        and the layer's block state that keeps the last of them."""
        T = h.shape[0]
        q, g, kv = self.in_proj.split(self.in_proj(h))
        native = ops.use_native(h)
        o = torch.empty(T, self.N, self.vdim, dtype=h.dtype, device=h.device)
        if kv_cache is None or md.is_dummy:
            o.zero_()
        else:
            (C if native else ref).latent_cache(kv, self.latent_norm, self.eps, kv_cache,
                                                md.slot_mapping, x, state, md.num_decode_tokens,
                                                md.cu_q_prefill)
            q_lat = torch.empty(T, self.N, self.W, dtype=h.dtype, device=h.device)
            torch.bmm(q.unflatten(1, (self.N, self.dim)).transpose(0, 1), self.w_uk,
                      out=q_lat.transpose(0, 1))
            o_lat = self._attend(q_lat, kv_cache, md)
            torch.bmm(o_lat.transpose(0, 1), self.w_uv, out=o.transpose(0, 1))
        o = (C if native else ref).sigmoid_gate(o.flatten(1), g)
        return self.o_proj(o)
