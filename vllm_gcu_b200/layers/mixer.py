"""Token mixers built from parts that read the same input and are summed.

A part (key attention, matrix memory, gated delta rule) names the projections it wants; a
``MixerBlock`` stacks those of all its parts into one GEMM, hands every part its views, and lets
the parts write their gated results side by side into one buffer that a single output GEMM sums.
A part's factor in the sum is applied when it writes, in 32-bit.  Projections whose results enter
a recurrence's gates unrounded come from a second, narrow GEMM with fp32 results; single tokens on
the GPU do without it (the parts' fused kernels take its weights).
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import ops
from ..ops import cuda as C
from ..parallel.state import tp_rank, tp_size
from .attention import AttentionMetadata
from .linear import MixedParallelLinear, MixedRowParallelLinear, linear_fp32

Projection = tuple[str, int, bool]      # name, output features, sharded over TP


def linear(x: torch.Tensor, weight: torch.Tensor, out: Optional[torch.Tensor] = None
           ) -> torch.Tensor:
    """``out``: where the rows go (a row-strided view is fine)."""
    if ops.use_native(x) and x.dtype == torch.bfloat16:
        return C.gemm_bf16(x, weight, out=out)
    y = F.linear(x, weight)
    return y if out is None else out.copy_(y)


class MixerPart(nn.Module):
    """``projections`` / ``fp32_projections`` / ``width`` (output features before the output
    projection, all ranks) are set by the constructor."""

    projections: Sequence[Projection]
    fp32_projections: Sequence[Projection] = ()
    width: int

    def new(self, *shape, dtype=torch.float32, device=None) -> nn.Parameter:
        return nn.Parameter(torch.zeros(shape, dtype=dtype, device=device), requires_grad=False)

    @staticmethod
    def shard(full: torch.Tensor, dim: int = 0) -> torch.Tensor:
        """This rank's slice of a tensor whose rows follow the heads."""
        return full.chunk(tp_size(), dim)[tp_rank()]

    def cache_shape(self) -> Optional[tuple[int, int]]:
        """(key / value heads, cached head dimension) if the part caches keys and values."""
        return None

    def state_shapes(self) -> dict:
        """Recurrent state per request: name -> (shape, dtype)."""
        return {}

    def load(self, name: str, full: torch.Tensor) -> bool:
        """Loads a tensor that is none of the projections; False if the part has no such one."""
        return False

    def own_tensors(self) -> set[str]:
        """Names that :meth:`load` takes."""
        return set()

    def mix(self, h: torch.Tensor, y: dict, f: dict, fw: dict, md: AttentionMetadata,
            cache: Optional[torch.Tensor], state: Optional[dict], scale: float, out: torch.Tensor
            ) -> None:
        """Writes ``scale`` times the part's result into ``out [T, local width]``.  ``y``: views of
        its projections of the mixer's input ``h`` (padded to multiples of 8 columns); ``f``: of its
        fp32 projections, without the rows of single tokens where :func:`fused_tokens` says so;
        ``fw``: the latter's weights."""
        raise NotImplementedError


def fused_tokens(h: torch.Tensor, md: AttentionMetadata) -> int:
    """Leading tokens of a step that fused single-token kernels take."""
    return md.num_decode_tokens if ops.use_native(h) and not md.is_dummy else 0


class MixerBlock(nn.Module):
    """``parts``: ``(checkpoint prefix, factor, part)``."""

    def __init__(self, parts: Sequence[tuple[str, float, MixerPart]], hidden: int, dtype, device,
                 prefix: str):
        super().__init__()
        self.names = [n for n, _, _ in parts]
        self.scales = [float(s) for _, s, _ in parts]
        self.parts = nn.ModuleList(p for _, _, p in parts)
        flat = [(i, *pr) for i, p in enumerate(self.parts) for pr in p.projections]
        self.slots = [(i, n) for i, n, _, _ in flat]
        self.in_proj = MixedParallelLinear(hidden, [s for _, _, s, _ in flat],
                                           [sh for _, _, _, sh in flat], dtype=dtype,
                                           device=device, prefix=prefix + ".in_proj", align=8)
        flat = [(i, *pr) for i, p in enumerate(self.parts) for pr in p.fp32_projections]
        self.fp32_slots = [(i, n) for i, n, _, _ in flat]
        self.fp32_proj = MixedParallelLinear(
            hidden, [s for _, _, s, _ in flat], [sh for _, _, _, sh in flat], dtype=dtype,
            device=device, prefix=prefix + ".fp32_proj", align=8) if flat else None
        self.o_proj = MixedRowParallelLinear([p.width for p in self.parts], hidden, dtype=dtype,
                                             device=device, prefix=prefix + ".o_proj")

    def cache_shape(self) -> Optional[tuple[int, int]]:
        shapes = [s for s in (p.cache_shape() for p in self.parts) if s is not None]
        assert len(shapes) <= 1, "one key / value cache per layer"
        return shapes[0] if shapes else None

    def state_shapes(self) -> dict:
        return {f"{i}.{k}": v for i, p in enumerate(self.parts)
                for k, v in p.state_shapes().items()}

    def load(self, name: str, full: torch.Tensor) -> bool:
        for i, (pre, part) in enumerate(zip(self.names, self.parts)):
            if not name.startswith(pre):
                continue
            sub = name[len(pre):]
            if (i, sub) in self.slots:
                self.in_proj.load_weight("weight", full, self.slots.index((i, sub)))
            elif (i, sub) in self.fp32_slots:
                self.fp32_proj.load_weight("weight", full, self.fp32_slots.index((i, sub)))
            elif sub == "o":
                self.o_proj.load_weight("weight", full, i)
            elif not part.load(sub, full):
                continue
            return True
        return False

    def tensor_names(self) -> set[str]:
        out = set()
        for i, (pre, part) in enumerate(zip(self.names, self.parts)):
            own = {n for j, n in self.slots + self.fp32_slots if j == i}
            out |= {pre + n for n in own | {"o"} | part.own_tensors()}
        return out

    def forward(self, h: torch.Tensor, md: AttentionMetadata, cache: Optional[torch.Tensor],
                state: Optional[dict]) -> torch.Tensor:
        T = h.shape[0]
        ys = self.in_proj.split(self.in_proj(h), padded=True)
        n1 = fused_tokens(h, md)
        fs, fws = (), ()
        if self.fp32_proj is not None:
            w = self.fp32_proj.weight
            fws = [v[:n] for v, n in zip(w.split(self.fp32_proj.padded_sizes),
                                         self.fp32_proj.local_sizes)]
            if n1 < T:
                fs = self.fp32_proj.split(linear_fp32(h[n1:], w))
        out = torch.empty(T, self.o_proj.in_per_rank, dtype=h.dtype, device=h.device)
        at = 0
        for i, part in enumerate(self.parts):
            y = {n: v for (j, n), v in zip(self.slots, ys) if j == i}
            f = {n: v for (j, n), v in zip(self.fp32_slots, fs) if j == i}
            fw = {n: v for (j, n), v in zip(self.fp32_slots, fws) if j == i}
            st = {k.partition(".")[2]: v for k, v in state.items()
                  if k.partition(".")[0] == str(i)} if state is not None else None
            w = self.o_proj.local_sizes[i]
            part.mix(h, y, f, fw, md, cache, st or None, self.scales[i], out[:, at:at + w])
            at += w
        return self.o_proj(out)
