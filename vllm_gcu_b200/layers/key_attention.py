"""Grouped attention over normalised queries and keys, as parts of a mixer.

* ``KeyAttention``: norm over the whole projection, rotary positions, attention sinks and an output
  gate; the values are the projected keys themselves.
* ``ChunkAttention``: norm over every head, no positions, soft capped scores, keys of the query's own
  chunk of positions only; values of their own, of any width.
* ``GroupedAttention``: what its ``AttentionSpec`` asks for of: norm over the whole projections,
  rotated halves with or without YaRN, a temperature of the queries by position, a norm of every
  head's values, values mixed with those of an earlier layer, learnt or zero sinks, a sliding window,
  a distance bias.

Paged cache ``[2, blocks, block_size, kv_heads, DC]`` as in ``PagedAttention``: normalised (rotated)
keys and values, heads padded to a width the tensor-core kernels take.  On the GPU one kernel
normalises, rotates and writes the cache; decode rows run through the split-KV kernels, portions
through the tcgen05 prefill kernel, everything else (32-bit models, wide heads, large groups)
through the general kernel of csrc/attention_any.cu.
"""
from __future__ import annotations

import math
from typing import Optional

import torch

from .. import ops
from ..config import AttentionSpec
from ..ops import cuda as C
from ..ops import ref
from ..parallel.communicator import get_comm
from ..parallel.state import tp_rank, tp_size
from .attention import AttentionMetadata
from .basic import RotaryEmbedding, build_cos_sin_cache
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
        self.register_buffer("slopes", None, persistent=False)

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
        rest = dict(scale=s.scale, sink=self.sink, softcap=s.softcap, chunk=s.chunk, out_dim=od,
                    window=s.window, slopes=self.slopes)
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
                most = min(n for n in (s.chunk, s.window, max(md.max_seq_len, 1)) if n > 0)
                if s.chunk or s.window:          # no more keys than a chunk or window holds
                    splits = min(splits, C.decode_num_splits(nd, self.G, most))
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


def rotary_table(spec: AttentionSpec, positions: int, device) -> Optional[torch.Tensor]:
    """fp32 ``[positions, rot_dims]`` cosines and sines of a ``GroupedAttention``, computed in fp64;
    None without rotation."""
    if not spec.rot_dims:
        return None
    scaling = None
    if spec.rot_scaling:
        factor, original, fast, slow = spec.rot_scaling
        scaling = {"type": "yarn", "factor": factor, "beta_fast": fast, "beta_slow": slow,
                   "original_max_position_embeddings": original,
                   "attention_factor": 0.1 * math.log(factor) + 1.0}
    return build_cos_sin_cache(spec.rot_dims, positions, spec.rot_base, scaling,
                               dtype=torch.float64).float().to(device)


def distance_slopes(num_heads: int) -> torch.Tensor:
    """2^(-8 (h + 1) / heads) for h = 0 .. heads - 1, for any number of heads (the sequence of
    ``alibi_slopes`` where that is a power of two)."""
    h = torch.arange(1, num_heads + 1, dtype=torch.float64)
    return torch.exp2(-8.0 * h / num_heads).float()


class GroupedAttention(CachedAttention):
    """``table``: see :func:`rotary_table`.  ``first``: the spec of the layer whose values this one
    mixes into its own (``AttentionMetadata.first_values`` is that layer's value cache), None in that
    layer itself or without mixing."""

    def __init__(self, spec: AttentionSpec, eps: float, dtype, device, prefix: str,
                 table: Optional[torch.Tensor], first: Optional[AttentionSpec] = None):
        super().__init__(spec, eps, dtype, prefix)
        H, G, D, VD = spec.num_heads, spec.num_kv_heads, spec.head_dim, self.VD
        if spec.rot_dims % 2 or not 0 <= spec.rot_dims <= D:
            raise ValueError(f"{prefix}: {spec.rot_dims} rotated of {D} dimensions")
        if spec.rot_dims and not spec.rot_halves or not spec.v_head_dim:
            raise ValueError(f"{prefix}: grouped attention rotates halves and has values of its own")
        if spec.temp_every < 1:
            raise ValueError(f"{prefix}: a temperature step every {spec.temp_every} positions")
        if first is not None and first.num_kv_heads * first.v_head_dim != G * VD:
            raise ValueError(f"{prefix}: {G} x {VD} values mixed with {first.num_kv_heads} x "
                             f"{first.v_head_dim}")
        self.projections = [("q", H * D, True), ("k", G * D, True), ("v", G * VD, True)]
        self.table, self.first = table, first          # shared by the layers, not a weight
        self._own = {}
        new = lambda *s: self.new(*s, device=device)  # noqa: E731
        self.q_norm = self.k_norm = None
        if spec.qk_norm:
            self.q_norm, self.k_norm = new(self.H * D), new(self.G * D)
            self._own.update({"q.norm": "q_norm", "k.norm": "k_norm"})
        if spec.sink == "learnt":
            self.sink = new(self.H)
            self._own["sink"] = "sink"
        elif spec.sink == "zero":
            self.sink = torch.zeros(self.H, dtype=torch.float32, device=device)
        if spec.v_mix:
            # (1 - share) * own + share * first; the first layer's is in checkpoints but unused
            self.share = new()
            self._own["vmix"] = "share"
        if spec.distance_bias:
            self.slopes = distance_slopes(H).view(tp_size(), -1)[tp_rank()].clone().to(device)

    def own_tensors(self) -> set[str]:
        return set(self._own)

    def load(self, name: str, full: torch.Tensor) -> bool:
        if name not in self._own:
            return False
        p = getattr(self, self._own[name])
        p.data.copy_(full.reshape(()) if name == "vmix" else self.shard(full))
        return True

    def mix(self, h, y, f, fw, md: AttentionMetadata, cache: Optional[torch.Tensor],
            state: Optional[dict], scale: float, out: torch.Tensor) -> None:
        s, D = self.spec, self.spec.head_dim
        if cache is None or md.is_dummy:
            out.zero_()
            return
        o_ = C if ops.use_native(out) else ref
        q, k = y["q"][:, :self.H * D], y["k"][:, :self.G * D]
        v = y["v"][:, :self.G * self.VD]
        tp, sumsq = tp_size(), None
        if tp > 1 and s.qk_norm:          # the norms run over the heads of all ranks
            sumsq = get_comm("tp").all_reduce(torch.stack(
                [q.float().pow(2).sum(-1), k.float().pow(2).sum(-1)], dim=1).contiguous())
        mixed = {} if self.first is None else dict(
            share=self.share, first=md.first_values, first_dim=self.first.v_head_dim)
        qn = o_.qkv_cache(q, k, v, self.q_norm, self.k_norm, self.eps, self.table, md.positions,
                          md.slot_mapping, cache[0], cache[1], D, self.VD, v_norm=s.v_norm,
                          temp=(s.temp_coef, s.temp_every), sumsq=sumsq, ranks=tp, **mixed)
        self._attend(qn, cache, md, out.unflatten(1, (self.H, self.VD)))
        if scale != 1.0:
            out.mul_(scale)
