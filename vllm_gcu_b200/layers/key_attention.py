"""Grouped attention over normalised queries and keys, as parts of a mixer.

* ``KeyAttention``: norm over the whole projection, rotary positions, attention sinks and an output
  gate; the values are the projected keys themselves.
* ``ChunkAttention``: norm over every head, no positions, soft capped scores, keys of the query's own
  chunk of positions only; values of their own, of any width.

Paged cache ``[2, blocks, block_size, kv_heads, DC]`` as in ``PagedAttention``: normalised (rotated)
keys and values, heads padded to a width the tensor-core kernels take.  On the GPU one kernel
normalises, rotates and writes the cache; decode rows run through the split-KV kernels, portions
through the tcgen05 prefill kernel, everything else (32-bit models, wide heads, large groups)
through the general kernel of csrc/attention_any.cu.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config import AttentionSpec
from ..ops import cuda as C
from ..ops import ref
from ..parallel.communicator import get_comm
from ..parallel.state import tp_size
from .attention import AttentionMetadata
from .basic import RotaryEmbedding
from .mixer import MixerPart

#: query heads per key head the decode kernels take
MAX_DECODE_GROUP = 16
MAX_HEAD_DIM = 512


def cached_head_dim(head_dim: int, dtype: torch.dtype) -> int:
    """Width of a cached head: one the tensor-core kernels cover where that is possible."""
    if dtype == torch.bfloat16:
        for n in (64, 96, 128):
            if head_dim <= n:
                return n
    return -(-head_dim // 4) * 4


class CachedAttention(MixerPart):
    """Heads, cache and attention kernels that the kinds of attention share."""

    def __init__(self, spec: AttentionSpec, eps: float, dtype, prefix: str):
        super().__init__()
        self.spec, self.eps = spec, eps
        H, G = spec.num_heads, spec.num_kv_heads
        self.VD = spec.v_head_dim or spec.head_dim
        widest = max(spec.head_dim, self.VD)
        tp = tp_size()
        if H % G:
            raise ValueError(f"{prefix}: {H} query heads over {G} key heads")
        if H % tp or G % tp:
            raise ValueError(f"{prefix}: {H} query and {G} key heads over {tp} ranks")
        if widest > MAX_HEAD_DIM:
            raise ValueError(f"{prefix}: heads of {widest} dimensions, at most {MAX_HEAD_DIM}")
        self.H, self.G, self.DC = H // tp, G // tp, cached_head_dim(widest, dtype)
        self.width = H * self.VD
        self.sink = None

    def cache_shape(self) -> tuple[int, int]:
        return self.G, self.DC

    _OWN: dict = {}

    def own_tensors(self) -> set[str]:
        return set(self._OWN)

    def _attend(self, q: torch.Tensor, cache: torch.Tensor, md: AttentionMetadata,
                out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``out``: rows ``[T, H, VD]`` (the row pitch is free) for the first VD columns of every
        head's result; None: all DC columns."""
        s = self.spec
        kc, vc = cache[0], cache[1]
        nd, npf, nr = md.num_decode_tokens, md.num_prefills, md.num_decodes
        od = self.DC if out is None else self.VD
        rest = dict(scale=s.scale, sink=self.sink, softcap=s.softcap, chunk=s.chunk, out_dim=od)
        if not ops.use_native(q):
            return ref.any_attention(q, kc, vc, md.block_tables, md.seq_lens, nd, md.cu_q_prefill,
                                     out=out, **rest)
        tensor_cores = q.dtype == torch.bfloat16 and self.DC in (64, 96, 128)
        if not tensor_cores:
            return C.any_attention(q, kc, vc, md.block_tables, md.seq_lens, nd, md.cu_q_prefill,
                                   out=out, **rest)
        if out is None:
            out = torch.empty_like(q)
        if nd > 0:
            if self.H // self.G <= MAX_DECODE_GROUP:
                splits = md.decode_splits
                if s.chunk:          # no more keys than a chunk holds
                    splits = min(splits, C.decode_num_splits(nd, self.G,
                                                             min(s.chunk, max(md.max_seq_len, 1))))
                C.paged_decode(q[:nd], kc, vc, md.block_tables[:nd], md.seq_lens[:nd], out=out[:nd],
                               num_splits=splits, workspace=md.decode_workspace, **rest)
            else:
                C.any_attention(q[:nd], kc, vc, md.block_tables[:nd], md.seq_lens[:nd], nd, None,
                                out=out[:nd], **rest)
        if npf > 0:
            bt, sl = md.block_tables[nr:nr + npf], md.seq_lens[nr:nr + npf]
            done = C.fmha_prefill_sink(q[nd:], kc, vc, bt, md.cu_q_prefill, sl, out=out[nd:],
                                       num_q_tiles_128=md.num_q_tiles_128, **rest)
            if done is None:
                C.any_attention(q[nd:], kc, vc, bt, sl, 0, md.cu_q_prefill, out=out[nd:], **rest)
        return out


class KeyAttention(CachedAttention):
    def __init__(self, spec: AttentionSpec, eps: float, dtype, device, prefix: str,
                 rotary: RotaryEmbedding):
        super().__init__(spec, eps, dtype, prefix)
        self.rotary = rotary
        H, G, D = spec.num_heads, spec.num_kv_heads, spec.head_dim
        if spec.rot_dims % 2 or not 0 <= spec.rot_dims <= D:
            raise ValueError(f"{prefix}: {spec.rot_dims} rotated of {D} dimensions")
        self.projections = [("q", H * D, True), ("k", G * D, True), ("g", H * D, True)]
        self.q_norm = self.new(self.H * D, device=device)
        self.k_norm = self.new(self.G * D, device=device)
        self.sink = self.new(self.H, device=device)

    _OWN = {"q.norm": "q_norm", "k.norm": "k_norm", "sink": "sink"}

    def load(self, name: str, full: torch.Tensor) -> bool:
        if name not in self._OWN:
            return False
        getattr(self, self._OWN[name]).data.copy_(self.shard(full))
        return True

    def mix(self, h, y, f, fw, md: AttentionMetadata, cache: Optional[torch.Tensor],
            state: Optional[dict], scale: float, out: torch.Tensor) -> None:
        D = self.spec.head_dim
        if cache is None or md.is_dummy:
            out.zero_()
            return
        o_ = C if ops.use_native(out) else ref
        q, k = y["q"][:, :self.H * D], y["k"][:, :self.G * D]
        tp, sumsq = tp_size(), None
        if tp > 1:          # the norm runs over the heads of all ranks
            sumsq = get_comm("tp").all_reduce(torch.stack(
                [q.float().pow(2).sum(-1), k.float().pow(2).sum(-1)], dim=1).contiguous())
        qn = o_.qk_norm_rope_cache(q, k, None, self.q_norm, self.k_norm, self.eps,
                                   self.rotary.cos_sin_cache, self.rotary.is_neox, md.positions,
                                   md.slot_mapping, cache[0], cache[1], D, sumsq, tp)
        o_.head_gate(self._attend(qn, cache, md), y["g"][:, :self.H * D], scale, D, out)


class ChunkAttention(CachedAttention):
    def __init__(self, spec: AttentionSpec, eps: float, dtype, device, prefix: str):
        super().__init__(spec, eps, dtype, prefix)
        H, G, D = spec.num_heads, spec.num_kv_heads, spec.head_dim
        if spec.rot_dims or not spec.v_head_dim:
            raise ValueError(f"{prefix}: chunked attention has no rotation and values of its own")
        self.projections = [("q", H * D, True), ("k", G * D, True), ("v", G * self.VD, True)]
        self.q_norm = self.new(D, device=device)
        self.k_norm = self.new(D, device=device)

    _OWN = {"q.norm": "q_norm", "k.norm": "k_norm"}

    def load(self, name: str, full: torch.Tensor) -> bool:
        if name not in self._OWN:
            return False
        getattr(self, self._OWN[name]).data.copy_(full)      # shared by the heads of all ranks
        return True

    def mix(self, h, y, f, fw, md: AttentionMetadata, cache: Optional[torch.Tensor],
            state: Optional[dict], scale: float, out: torch.Tensor) -> None:
        D = self.spec.head_dim
        if cache is None or md.is_dummy:
            out.zero_()
            return
        o_ = C if ops.use_native(out) else ref
        qn = o_.head_norm_cache(y["q"][:, :self.H * D], y["k"][:, :self.G * D],
                                y["v"][:, :self.G * self.VD], self.q_norm, self.k_norm, self.eps,
                                md.slot_mapping, cache[0], cache[1], D)
        self._attend(qn, cache, md, out.unflatten(1, (self.H, self.VD)))
        if scale != 1.0:
            out.mul_(scale)
