"""Mixer parts with a matrix state per head: gated delta rule, matrix memory and time mixing.

Their state belongs to a request, not to its cache blocks: it lives in the request's state slot
(``AttentionMetadata.state_slots``) in fp32 and is updated in place by every step.  A portion at
position 0 starts from zeros, so slots are handed on without clearing.  See csrc/recurrent.cu for
the layout.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn as nn

from .. import ops
from ..config import DeltaSpec, MemorySpec, TimeMixSpec
from ..ops import cuda as C
from ..ops import ref
from ..parallel.state import tp_size
from .attention import AttentionMetadata
from .linear import MixedParallelLinear, ReplicatedLinear, RowParallelLinear, linear_fp32
from .mixer import MixerPart, fused_tokens, linear

#: padded key dimensions of the scan kernel
STATE_ROWS = (32, 64, 96, 128, 192, 256)
MAX_TAPS = 8


@dataclass
class Place:
    """What the scans need to know of a step (or of its rows behind the single tokens)."""
    positions: torch.Tensor
    state_slots: Optional[torch.Tensor]
    num_decode_tokens: int
    cu_q_prefill: Optional[torch.Tensor]

    @staticmethod
    def behind(md: AttentionMetadata, n: int) -> "Place":
        """``n``: 0 or all single tokens of the step (one request each)."""
        slots = md.state_slots[n:] if md.state_slots is not None else None
        return Place(md.positions[n:], slots, md.num_decode_tokens - n, md.cu_q_prefill)


def state_rows(head_dim: int, prefix: str) -> int:
    for n in STATE_ROWS:
        if head_dim <= n:
            return n
    raise ValueError(f"{prefix}: a state with {head_dim} keys per head, at most {STATE_ROWS[-1]}")


def _local_heads(heads: int, prefix: str) -> int:
    tp = tp_size()
    if heads % tp:
        raise ValueError(f"{prefix}: {heads} heads over {tp} ranks")
    return heads // tp


class GatedDelta(MixerPart):
    """Gated delta rule with one decay per head and key channel.  Queries, keys and values pass a
    short causal convolution and SiLU; decays and the output gate come from two-step projections."""

    def __init__(self, spec: DeltaSpec, eps: float, dtype, device, prefix: str):
        super().__init__()
        self.spec, self.eps, self.dtype = spec, eps, dtype
        N, G, D, V = spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.v_head_dim
        if N % G:
            raise ValueError(f"{prefix}: {N} heads over {G} query / key heads")
        if not 1 <= spec.conv_taps <= MAX_TAPS:
            raise ValueError(f"{prefix}: a convolution of {spec.conv_taps} taps, at most "
                             f"{MAX_TAPS}")
        self.N, self.G = _local_heads(N, prefix), _local_heads(G, prefix)
        self.rows = state_rows(D, prefix)
        self.width = N * V
        self.projections = [("q", G * D, True), ("k", G * D, True), ("v", N * V, True),
                            ("a1", spec.decay_rank, False), ("g1", spec.gate_rank, False)]
        self.fp32_projections = [("b", N, True)]
        new = lambda *s, dt=torch.float32: self.new(*s, dtype=dt, device=device)  # noqa: E731
        self.conv_q, self.conv_k = (new(spec.conv_taps, self.G * D) for _ in range(2))
        self.conv_v = new(spec.conv_taps, self.N * V)
        self.a_log, self.dt_bias = new(self.N), new(self.N * D)
        self.norm = new(V)
        pad = lambda n: -(-n // 8) * 8  # noqa: E731
        self.a2 = new(self.N * D, pad(spec.decay_rank), dt=dtype)      # columns behind the rank
        self.g2 = new(self.N * V, pad(spec.gate_rank), dt=dtype)       # stay zero

    def state_shapes(self) -> dict:
        s = self.spec
        C_ = 2 * self.G * s.head_dim + self.N * s.v_head_dim
        return {"matrix": ((self.N, s.v_head_dim, self.rows), torch.float32),
                "taps": ((s.conv_taps, C_), self.dtype)}

    _OWN = {"q.conv": "conv_q", "k.conv": "conv_k", "v.conv": "conv_v", "A_log": "a_log",
            "dt_bias": "dt_bias", "norm": "norm", "a2": "a2", "g2": "g2"}

    def own_tensors(self) -> set[str]:
        return set(self._OWN)

    def load(self, name: str, full: torch.Tensor) -> bool:
        if name not in self._OWN:
            return False
        p = getattr(self, self._OWN[name]).data
        t = full if name == "norm" else self.shard(full)
        if name.endswith(".conv"):
            t = t.t()
        (p[:, :t.shape[1]] if name in ("a2", "g2") else p).copy_(t)
        return True

    def finalize(self) -> None:
        self.a2.data[:, self.spec.decay_rank:] = 0
        self.g2.data[:, self.spec.gate_rank:] = 0

    def mix(self, h, y, f, fw, md: AttentionMetadata, cache, state: Optional[dict], scale: float,
            out: torch.Tensor) -> None:
        s = self.spec
        nk, nv = self.G * s.head_dim, self.N * s.v_head_dim
        q, k, v, a1, g1 = y["q"][:, :nk], y["k"][:, :nk], y["v"][:, :nv], y["a1"], y["g1"]
        conv = (self.conv_q, self.conv_k, self.conv_v)
        sizes = s.head_dim, s.v_head_dim, self.rows
        z, gate = linear_fp32(a1, self.a2), linear(g1, self.g2)
        n1 = fused_tokens(h, md)
        if n1:
            C.delta_step(h[:n1], q[:n1], k[:n1], v[:n1], z[:n1], gate[:n1], fw["b"], conv,
                         self.dt_bias, self.a_log, self.norm, *sizes, md.positions,
                         md.state_slots, state, self.eps, scale, out[:n1])
        if n1 == h.shape[0]:
            return
        o_ = C if ops.use_native(out) else ref
        o = o_.delta_rule(q[n1:], k[n1:], v[n1:], z[n1:], f["b"], conv, self.dt_bias, self.a_log,
                          *sizes, Place.behind(md, n1), None if md.is_dummy else state)
        o_.head_norm_gate(o, self.norm, gate[n1:], self.eps, scale, out[n1:])


class MatrixMemory(MixerPart):
    """Matrix memory of an mLSTM: exponential input gate, forget gate in log space, a running
    maximum that keeps both in range, and a normaliser vector."""

    def __init__(self, spec: MemorySpec, eps: float, dtype, device, prefix: str):
        super().__init__()
        self.spec, self.eps = spec, eps
        N, D, V = spec.num_heads, spec.head_dim, spec.v_head_dim
        self.N = _local_heads(N, prefix)
        self.rows = state_rows(D, prefix)
        self.width = N * V
        self.projections = [("q", N * D, True), ("k", N * D, True), ("v", N * V, True),
                            ("g", N * V, True)]
        self.fp32_projections = [("i", N, True), ("f", N, True)]
        self.i_bias, self.f_bias = self.new(self.N, device=device), self.new(self.N, device=device)
        self.norm = self.new(self.N * V, device=device)

    def state_shapes(self) -> dict:
        f32 = torch.float32
        return {"matrix": ((self.N, self.spec.v_head_dim, self.rows), f32),
                "vector": ((self.N, self.rows), f32), "scalar": ((self.N,), f32)}

    _OWN = {"i.b": "i_bias", "f.b": "f_bias", "norm": "norm"}

    def own_tensors(self) -> set[str]:
        return set(self._OWN)

    def load(self, name: str, full: torch.Tensor) -> bool:
        if name not in self._OWN:
            return False
        getattr(self, self._OWN[name]).data.copy_(self.shard(full))
        return True

    def mix(self, h, y, f, fw, md: AttentionMetadata, cache, state: Optional[dict], scale: float,
            out: torch.Tensor) -> None:
        s = self.spec
        nk, nv = self.N * s.head_dim, self.N * s.v_head_dim
        q, k, v, g = y["q"][:, :nk], y["k"][:, :nk], y["v"][:, :nv], y["g"][:, :nv]
        sizes = s.head_dim, s.v_head_dim, self.rows
        n1 = fused_tokens(h, md)
        if n1:
            C.memory_step(h[:n1], q[:n1], k[:n1], v[:n1], g[:n1], fw["i"], fw["f"], self.i_bias,
                          self.f_bias, s.gate_cap, self.norm, *sizes, md.positions,
                          md.state_slots, state, self.eps, scale, out[:n1])
        if n1 == h.shape[0]:
            return
        o_ = C if ops.use_native(out) else ref
        o, nq, low = o_.matrix_memory(q[n1:], k[n1:], v[n1:], f["i"], f["f"], self.i_bias,
                                      self.f_bias, s.gate_cap, *sizes, Place.behind(md, n1),
                                      None if md.is_dummy else state)
        o_.head_norm_gate(o, self.norm, g[n1:], self.eps, scale, out[n1:], nq, low)


class TimeMix(nn.Module):
    """Linear recurrence of the RWKV kind: a matrix per head that decays per key channel, and a bonus
    for the current token.

    A mixer of its own (not a part of a ``MixerBlock``): its five projections (r, k, v, the output
    gate g, the decay's first step w) read five different mixtures of a token's row with the row of
    the token before it, which come from the input convolution's kernel as ``h [5, T, H]``, in the
    order of ``MIXES`` (``layers/input_conv.py``)."""

    MIXES = ("r", "k", "v", "g", "w")

    def __init__(self, spec: TimeMixSpec, hidden: int, eps: float, dtype, device, prefix: str):
        super().__init__()
        self.spec, self.eps, self.dtype = spec, eps, dtype
        N, D, R = spec.num_heads, spec.head_dim, spec.decay_rank
        self.N = _local_heads(N, prefix)
        self.rows = state_rows(D, prefix)
        new = lambda *s, dt=torch.float32: nn.Parameter(  # noqa: E731
            torch.zeros(*s, dtype=dt, device=device), requires_grad=False)
        self.mu = new(len(self.MIXES), hidden)
        self.in_proj = MixedParallelLinear(hidden, [N * D] * 4, [True] * 4, dtype=dtype,
                                           device=device, prefix=prefix + ".in_proj", align=8)
        pad = -(-R // 8) * 8
        self.w1 = ReplicatedLinear(hidden, pad, dtype=dtype, device=device, prefix=prefix + ".w1")
        self.w2 = new(self.N * D, pad, dt=dtype)           # columns behind the rank stay zero
        self.w0, self.bonus = new(self.N * D), new(self.N * D)
        self.norm = new(self.N * D)
        self.o_proj = RowParallelLinear(N * D, hidden, dtype=dtype, device=device,
                                        prefix=prefix + ".o_proj")
        # few rows: the four projections as one grouped product, a tile of rows each
        self.tiles = self.tile_rows = None
        if self.in_proj.weight.is_cuda and dtype == torch.bfloat16 and hidden % 8 == 0 \
                and self.in_proj.padded_sizes[0] % 64 == 0:
            self.tiles = torch.arange(4, dtype=torch.int32, device=device)
            self.tile_rows = torch.tensor([4 * C.GROUP_ROWS], dtype=torch.int32, device=device)

    def cache_shape(self) -> None:
        return None

    def state_shapes(self) -> dict:
        """Recurrent state per request: name -> (shape, dtype)."""
        return {"matrix": ((self.N, self.spec.head_dim, self.rows), torch.float32)}

    _OWN = {"w0": "w0", "u": "bonus", "norm": "norm"}

    def tensor_names(self) -> set[str]:
        return {"mu." + c for c in self.MIXES} | {"r", "k", "v", "g", "w1", "w2", "o"} | set(self._OWN)

    def load(self, name: str, full: torch.Tensor) -> bool:
        """False if there is no tensor of that name."""
        if name not in self.tensor_names():
            return False
        if name.startswith("mu."):
            self.mu.data[self.MIXES.index(name[3:])].copy_(full)
        elif name == "w1":
            self.w1.weight.data[:self.spec.decay_rank].copy_(full)
        elif name == "w2":
            self.w2.data[:, :self.spec.decay_rank].copy_(MixerPart.shard(full))
        elif name == "o":
            self.o_proj.load_weight("weight", full)
        elif name in self._OWN:
            getattr(self, self._OWN[name]).data.copy_(MixerPart.shard(full.reshape(-1)))
        else:
            self.in_proj.load_weight("weight", full, self.MIXES.index(name))
        return True

    def finalize(self) -> None:
        self.w1.weight.data[self.spec.decay_rank:] = 0
        self.w2.data[:, self.spec.decay_rank:] = 0

    def _project(self, h: torch.Tensor, n: int) -> list[torch.Tensor]:
        """r, k, v and the gate ``[T, n]``, views of equal row pitch."""
        T, pad, w = h.shape[1], self.in_proj.padded_sizes[0], self.in_proj.weight
        if self.tiles is not None and T <= C.GROUP_ROWS \
                and h.stride(0) == C.GROUP_ROWS * h.shape[2]:
            y = C.gemm_bf16_grouped(h.as_strided((4 * C.GROUP_ROWS, h.shape[2]), (h.stride(1), 1)),
                                    w.view(4, pad, -1), self.tiles, self.tile_rows)
            return [y[i * C.GROUP_ROWS:i * C.GROUP_ROWS + T, :n] for i in range(4)]
        y = torch.empty(T, 4 * pad, dtype=h.dtype, device=h.device)
        for i in range(4):
            linear(h[i], w[i * pad:(i + 1) * pad], out=y[:, i * pad:(i + 1) * pad])
        return [y[:, i * pad:i * pad + n] for i in range(4)]

    def forward(self, h: torch.Tensor, md: AttentionMetadata, state: Optional[dict]) -> torch.Tensor:
        T, D, n = h.shape[1], self.spec.head_dim, self.N * self.spec.head_dim
        r, k, v, g = self._project(h, n)
        a = linear_fp32(h[4], self.w1.weight)              # the decay's inner row, unrounded
        out = torch.empty(T, n, dtype=h.dtype, device=h.device)
        S = state["matrix"] if state is not None and not md.is_dummy else None
        n1 = fused_tokens(h, md)
        if n1:
            C.wkv_step(r[:n1], k[:n1], v[:n1], g[:n1], a[:n1], self.w2, self.w0, self.bonus,
                       self.norm, D, self.rows, md.positions, md.state_slots, S, self.eps, out[:n1])
        if n1 < T:
            o_ = C if ops.use_native(out) else ref
            z = linear_fp32(o_.tanh_rows(a[n1:], self.dtype), self.w2)
            o = o_.wkv(r[n1:], k[n1:], v[n1:], z, self.w0, self.bonus, D, self.rows,
                       Place.behind(md, n1), S)
            o_.head_norm_gate(o, self.norm, g[n1:], self.eps, 1.0, out[n1:], act="silu")
        return self.o_proj(out)
