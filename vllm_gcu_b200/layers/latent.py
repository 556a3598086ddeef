"""Latent attention with or without a rotated part, and the token shift some designs put in front.

``LatentAttention`` caches one normalised latent row per token.  Keys and values of every head
are linear in that row, so they are absorbed: the query is carried into latent space with W_uk,
attention runs over the cached rows themselves (all heads share them), and W_uv expands the
result.  Queries, output gate and latent come from one GEMM.  Steps on the GPU:

1. ``in_proj``: ``[q | gate | latent, rotated key part]`` of the step's rows;
2. ``q W_uk``;
3. one kernel normalises the latent into the paged cache (rows padded with zeros to the tile
   width of the attention kernel), rotates the key part into the columns behind it and the query
   parts into the same columns of the latent queries, and keeps the rows that a token shift needs
   later;
4. attention (tcgen05 kernel where the layout allows, csrc/attention_mla.cu, else
   csrc/latent.cu), with a sink per head in the denominator and the gate of a head on its result
   where the design has them; ``o W_uv``;
5. output gate per channel if the design has that kind, ``o_proj``.

The rotated columns follow the latent without a gap.  The value part of a cached row is rounded up to
whole tiles and may reach into them: W_uv has zero rows there.

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


def latent_row_width(kv_rank: int, dtype: torch.dtype, rot_dim: int = 0) -> int:
    """Columns of a cached latent row: whole 64-column tiles where the tcgen05 kernel takes the
    layout, else a multiple of four."""
    n = kv_rank + rot_dim
    if dtype == torch.bfloat16 and kv_rank <= 512 and n <= 576:
        return -(-n // 64) * 64
    return -(-n // 4) * 4


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
    """``cos_sin``: fp32 table ``[positions, rot_dim]`` of a design with a rotated part."""

    def __init__(self, spec: LayerSpec, hidden: int, eps: float, dtype, device, prefix: str,
                 cos_sin: Optional[torch.Tensor] = None):
        super().__init__()
        tp = tp_size()
        if spec.num_heads % tp:
            raise ValueError(f"{prefix}: {spec.num_heads} heads over {tp} ranks")
        if spec.rot_dim % 2:
            raise ValueError(f"{prefix}: {spec.rot_dim} rotated dimensions do not pair up")
        self.N, self.dim, self.vdim = spec.num_heads // tp, spec.head_dim, spec.v_head_dim
        self.L, self.R, self.scale, self.eps = spec.kv_lora_rank, spec.rot_dim, spec.scale, eps
        self.W = latent_row_width(self.L, dtype, self.R)
        self.V = min(self.W, -(-self.L // 64) * 64)     # columns that the tcgen05 kernel sums
        self.cos_sin = cos_sin if self.R else None      # shared by the layers, not a weight
        self.head_gate = spec.head_gate
        A = spec.num_heads
        self.in_proj = MixedParallelLinear(
            hidden, [A * (self.dim + self.R), A if self.head_gate else A * self.vdim,
                     self.L + self.R], [True, True, False], dtype=dtype, device=device,
            prefix=prefix + ".in_proj", align=8)
        new = lambda *s: nn.Parameter(torch.zeros(*s, dtype=dtype, device=device),  # noqa: E731
                                      requires_grad=False)
        self.latent_norm = new(self.L)
        self.w_uk = new(self.N, self.dim, self.W)       # columns behind L stay zero
        self.w_uv = new(self.N, self.W, self.vdim)      # rows behind L stay zero
        self.sink = nn.Parameter(torch.zeros(self.N, dtype=torch.float32, device=device),
                                 requires_grad=False) if spec.sink else None
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
        elif name == "sink" and self.sink is not None:
            self.sink.data.copy_(full[r * N:(r + 1) * N])
        else:
            raise KeyError(name)

    def load(self, name: str, full: torch.Tensor) -> bool:
        """False if there is no tensor of that name."""
        if name not in self.tensor_names():
            return False
        self.load_weight(name, full)
        return True

    def tensor_names(self) -> set[str]:
        return {"q", "g", "dkv", "dkv.norm", "uk", "uv", "o"} | (
            {"sink"} if self.sink is not None else set())

    def finalize(self) -> None:
        self.w_uk.data[:, :, self.L:] = 0
        self.w_uv.data[:, self.L:] = 0

    def _attend(self, q: torch.Tensor, cache: torch.Tensor, md: AttentionMetadata,
                gate: Optional[torch.Tensor]) -> torch.Tensor:
        """Causal attention of latent queries ``[T, N, W]`` over the cached rows."""
        T, nd = q.shape[0], md.num_decode_tokens
        rest = dict(sink=self.sink, gate=gate)
        if not ops.use_native(q):
            ql = [1] * md.num_decodes + list(md.q_lens_cpu[md.num_decodes:])
            return ref.latent_attention(q, cache, md.block_tables, ql, md.seq_lens_cpu, self.scale,
                                        self.W, **rest)
        if not C.mla_attention_supported(q, cache, self.V):
            return C.latent_attention(q, cache, md.block_tables, md.seq_lens, nd, md.cu_q_prefill,
                                      self.scale, **rest)
        out = torch.empty(T, self.N, self.V, dtype=q.dtype, device=q.device)
        max_len = max(md.max_seq_len, 1)

        def part(lo: int, hi: int, first: int, end: int, cu_q, tiles: int) -> None:
            if gate is not None:
                rest["gate"] = gate[lo:hi]
            C.mla_attention(q[lo:hi], cache, md.block_tables[first:end], md.seq_lens[first:end],
                            cu_q, tiles, max_len, self.scale, out=out[lo:hi], L=self.V, **rest)
        if nd > 0:
            part(0, nd, 0, nd, None, nd)
        if md.num_prefills > 0:
            B = md.num_decodes + md.num_prefills
            tq = 128 // self.N
            ql = md.q_lens_cpu[md.num_decodes:B]
            n = sum(ql)
            part(nd, nd + n, md.num_decodes, B, md.cu_q_prefill, sum(-(-x // tq) for x in ql))
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
        o_ = C if ops.use_native(h) else ref
        o = torch.empty(T, self.N, self.vdim, dtype=h.dtype, device=h.device)
        if kv_cache is None or md.is_dummy:
            o.zero_()
        else:
            q_lat = torch.empty(T, self.N, self.W, dtype=h.dtype, device=h.device)
            torch.bmm(q.unflatten(1, (self.N, -1))[..., :self.dim].transpose(0, 1), self.w_uk,
                      out=q_lat.transpose(0, 1))
            rot = dict(cos_sin=self.cos_sin, positions=md.positions, q=q, q_lat=q_lat) \
                if self.R else {}
            o_.latent_cache(kv, self.latent_norm, self.eps, kv_cache, md.slot_mapping, x, state,
                            md.num_decode_tokens, md.cu_q_prefill, **rot)
            o_lat = self._attend(q_lat, kv_cache, md, g if self.head_gate else None)
            torch.bmm(o_lat.transpose(0, 1), self.w_uv[:, :o_lat.shape[2]],
                      out=o.transpose(0, 1))
        o = o.flatten(1)
        return self.o_proj(o if self.head_gate else o_.sigmoid_gate(o, g))
