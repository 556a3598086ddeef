"""Causal convolution in front of a mixer: ``h + conv(h)`` per channel, and the mixtures of a row with
the row before it that time mixing reads.

What a step needs of earlier ones is a request's last rows ``h`` (in the model's type): ``taps - 1``,
or ``taps`` where the convolved row of the token before is needed too (it is computed again from
them).  They live in the request's state slot as a ring indexed by position, read and written only by
the threads that hold the first rows of a request's portion, so slots are handed on without clearing
and a portion may have any length.

Single tokens on the GPU are convolved by the norm kernel that produces their row
(``ops.cuda.add_group_norm``), portions by a kernel of their own (``ops.cuda.input_conv``).
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from .. import ops
from ..ops import cuda as C
from ..ops import ref
from .attention import AttentionMetadata
from .mixer import fused_tokens
from .recurrent import MAX_TAPS, Place


class InputConv(nn.Module):
    """``mu [M, H]`` (fp32, or None): the mixtures ``c + (c' - c) * mu_m`` of a convolved row c with
    the one before it take the place of the row, ``[M, T, H]`` in all."""

    def __init__(self, hidden: int, taps: int, dtype, device, prefix: str,
                 mu: Optional[nn.Parameter] = None):
        super().__init__()
        if not 1 <= taps <= MAX_TAPS:
            raise ValueError(f"{prefix}: a convolution of {taps} taps, at most {MAX_TAPS}")
        self.hidden, self.taps, self.dtype = hidden, taps, dtype
        self.back = taps if mu is not None else taps - 1
        self.weight = nn.Parameter(torch.zeros(taps, hidden, dtype=torch.float32, device=device),
                                   requires_grad=False)
        object.__setattr__(self, "mu", mu)            # the mixer's parameter, not one of this module

    def state_shapes(self) -> dict:
        return {"inputs": ((self.back, self.hidden), self.dtype)} if self.back else {}

    def load_weight(self, name: str, full: torch.Tensor, shard_id=None) -> None:
        self.weight.data.copy_(full.t())

    def after_norm(self, norm, rows: torch.Tensor, md: AttentionMetadata, state: Optional[dict]
                   ) -> torch.Tensor:
        """``norm(lo, conv)`` runs the norm kernel: into ``lo [T, H]``, or for the leading single
        tokens through the convolution ``conv`` names.  Returns ``[T, H]`` or ``[M, T, H]`` like
        ``rows [T, H]`` in the model's type."""
        T = rows.shape[0]
        new = lambda *s: torch.empty(*s, dtype=self.dtype, device=rows.device)  # noqa: E731
        if self.mu is None:
            out = new(T, self.hidden)
        else:       # few rows: every mixture in a tile of rows of its own, as grouped products take it
            out = new(self.mu.shape[0], max(T, C.GROUP_ROWS) if rows.is_cuda else T,
                      self.hidden)[:, :T]
        ring = state["inputs"] if state is not None and self.back and not md.is_dummy else None
        n1 = fused_tokens(rows, md)
        lo = new(T, self.hidden)
        conv = (self.weight, self.mu, md.positions, md.state_slots, ring, out, n1) if n1 else None
        norm(lo, conv)
        if n1 < T:
            op = C.input_conv if ops.use_native(rows) else ref.input_conv
            op(lo[n1:], self.weight, self.mu, Place.behind(md, n1), ring, out[..., n1:, :])
        return out
