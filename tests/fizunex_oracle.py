"""Plain, slow evaluation of the Fizunex design in torch, one function per mechanism.

Test oracle only: whole sequences, no cache, no batching, nothing shared with the package.  All
functions take and return tensors of the dtype they are given (float32 or float64).

Notation: ``x`` is the residual stream ``[T, H]`` of one sequence, ``h`` a mixer's input, ``w``
maps tensor names to tensors.  A recurrence is a loop over tokens that holds one matrix per head.
"""
from __future__ import annotations

import math

import torch


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-torch.abs(z)))


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last dimension (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps: float) -> torch.Tensor:
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * weight + bias


def rotate_pairs(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """``x [T, heads, dim]`` at positions 0 .. T-1; neighbouring coordinates form the pairs, the
    coordinates from ``dims`` on pass."""
    out = x.clone()
    for p in range(x.shape[0]):
        for i in range(dims // 2):
            a = p * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[p, :, 2 * i], x[p, :, 2 * i + 1]
            out[p, :, 2 * i] = u * c - v * s
            out[p, :, 2 * i + 1] = v * c + u * s
    return out


def sink_softmax(scores: torch.Tensor, sink) -> torch.Tensor:
    """Weights over the last dimension with one more term exp(sink) in the denominator."""
    top = torch.maximum(scores.max(dim=-1, keepdim=True).values, sink)
    e = torch.exp(scores - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def key_value_attention(h: torch.Tensor, w: dict, heads: int, kv_heads: int, dim: int, rot_dims: int,
                        rot_base: float, scale: float, eps: float) -> torch.Tensor:
    """Causal attention whose values are the projected keys (before their norm and rotation).
    ``w``: q, k, q.norm, k.norm, sink, g, o."""
    T = h.shape[0]
    q, k = h @ w["q"].T, h @ w["k"].T
    v = k.view(T, kv_heads, dim)
    q = (rms_unit(q, eps) * w["q.norm"]).view(T, heads, dim)
    k = (rms_unit(k, eps) * w["k.norm"]).view(T, kv_heads, dim)
    q, k = rotate_pairs(q, rot_dims, rot_base), rotate_pairs(k, rot_dims, rot_base)
    ahead = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    out = torch.zeros(T, heads, dim, dtype=h.dtype)
    for a in range(heads):
        b = a // (heads // kv_heads)
        s = ((q[:, a] @ k[:, b].T) * scale).masked_fill(ahead, -math.inf)
        out[:, a] = sink_softmax(s, w["sink"][a]) @ v[:, b]
    return (out.reshape(T, heads * dim) * sigmoid(h @ w["g"].T)) @ w["o"].T


def memory_gates(zi, zf, cap: float):
    """Log input and log forget gate from their projections (bias included)."""
    soft = cap * torch.tanh(zf / cap)
    return cap * torch.tanh(zi / cap), -softplus(-soft)


def matrix_memory(q, k, v, i, f):
    """``q, k [T, heads, dim]`` (q already scaled), ``v [T, heads, vdim]``, log gates ``[T, heads]``
    -> ``[T, heads, vdim]``."""
    T, N, D = k.shape
    out = torch.zeros_like(v)
    for a in range(N):
        S = torch.zeros(D, v.shape[2], dtype=v.dtype)
        n = torch.zeros(D, dtype=v.dtype)
        m = torch.zeros((), dtype=v.dtype)
        for t in range(T):
            new = torch.maximum(f[t, a] + m, i[t, a])
            keep, add = torch.exp(f[t, a] + m - new), torch.exp(i[t, a] - new)
            S = keep * S + add * torch.outer(k[t, a], v[t, a])
            n = keep * n + add * k[t, a]
            m = new
            den = torch.maximum((n @ q[t, a]).abs(), torch.exp(-m)) + 1e-6
            out[t, a] = (S.T @ q[t, a]) / den
    return out


def matrix_memory_mixer(h, w: dict, heads: int, dim: int, vdim: int, cap: float, eps: float):
    """``w``: q, k, v, g, o, norm, i, i.b, f, f.b."""
    T = h.shape[0]
    q = (h @ w["q"].T).view(T, heads, dim) * dim ** -0.5
    k, v = (h @ w["k"].T).view(T, heads, dim), (h @ w["v"].T).view(T, heads, vdim)
    i, f = memory_gates(h @ w["i"].T + w["i.b"], h @ w["f"].T + w["f.b"], cap)
    o = rms_unit(matrix_memory(q, k, v, i, f), eps).reshape(T, heads * vdim)
    return (o * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def short_conv(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """Causal convolution per channel: ``x [T, C]``, ``taps [C, n]``, the last tap meets the
    current row, rows before the first are zero."""
    n = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            if t - (n - 1 - j) >= 0:
                out[t] += taps[:, j] * x[t - (n - 1 - j)]
    return out


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """``q, k [T, kv_heads, dim]``, ``v [T, heads, vdim]``, decays ``g [T, heads, dim]``, step sizes
    ``beta [T, heads]`` -> ``[T, heads, vdim]``."""
    T, N, _ = v.shape
    group = N // k.shape[1]
    out = torch.zeros_like(v)
    for a in range(N):
        b = a // group
        S = torch.zeros(k.shape[2], v.shape[2], dtype=v.dtype)
        for t in range(T):
            S = g[t, a][:, None] * S
            u = beta[t, a] * (v[t, a] - S.T @ k[t, b])
            S = S + torch.outer(k[t, b], u)
            out[t, a] = S.T @ q[t, b]
    return out


def channel_delta_mixer(h, w: dict, heads: int, kv_heads: int, dim: int, vdim: int, eps: float):
    """``w``: q, k, v and their .conv, b, A_log, a1, a2, dt_bias, g1, g2, norm, o."""
    T = h.shape[0]
    q, k, v = (silu(short_conv(h @ w[c].T, w[c + ".conv"])) for c in ("q", "k", "v"))
    q = unit(q.view(T, kv_heads, dim)) * dim ** -0.5
    k = unit(k.view(T, kv_heads, dim))
    v = v.view(T, heads, vdim)
    step = softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).view(T, heads, dim)
    g = torch.exp(-torch.exp(w["A_log"])[None, :, None] * step)
    o = delta_rule(q, k, v, g, sigmoid(h @ w["b"].T))
    o = rms_unit(o, eps) * w["norm"]
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T)
    return (o.reshape(T, heads * vdim) * gate) @ w["o"].T


def dense(h, w: dict):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def sub(w: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def mixer(h, layer: dict, w: dict, eps: float):
    m = layer["mixer"]
    if layer["type"] == "channel_delta":
        return channel_delta_mixer(h, w, m["heads"], m["kv_heads"], m["dim"], m["vdim"], eps)
    a, b = m["left"], m["right"]
    left = key_value_attention(h, sub(w, "left."), a["heads"], a["kv_heads"], a["dim"],
                               a["rot"]["dims"], a["rot"]["base"], a["scale"], eps)
    right = matrix_memory_mixer(h, sub(w, "right."), b["heads"], b["dim"], b["vdim"],
                                b["gate_cap"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


def run_layers(config: dict, weights: dict, tokens, dtype=torch.float64) -> list:
    """Residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * config["embedding"]["scale"]
    out = []
    for i, layer in enumerate(config["layers"]):
        lw = sub(w, f"l{i}.")
        x = x + layer_norm(mixer(x, layer, sub(lw, "mix."), eps), lw["norm1"], lw["norm1.b"], eps)
        if layer["mlp"] is not None:
            x = x + layer_norm(dense(x, sub(lw, "mlp.")), lw["norm2"], lw["norm2.b"], eps)
        out.append(x)
    return out


def forward(config: dict, weights: dict, tokens, dtype=torch.float64) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence."""
    x = run_layers(config, weights, tokens, dtype)[-1]
    w = {k: weights[k].to(dtype) for k in ("embed", "final.norm", "final.norm.b")}
    x = layer_norm(x, w["final.norm"], w["final.norm.b"], config["norm"]["eps"])
    return (x @ w["embed"].T) * config["logit_scale"]


def tensor_shapes(config: dict, ranks=(5, 7)) -> dict:
    """Names and shapes of all tensors; ``ranks`` of the decay's and the gate's two-step
    projections (no number of the configuration)."""
    H = config["width"]
    s = {"embed": (config["vocab"], H), "final.norm": (H,), "final.norm.b": (H,)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for n in ("norm1", "norm2") if layer["mlp"] is not None else ("norm1",):
            s[p + n] = s[p + n + ".b"] = (H,)
        p += "mix."
        if layer["type"] == "channel_delta":
            N, G, D, V, c = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, r in (("q", G * D), ("k", G * D), ("v", N * V)):
                s[p + n], s[p + n + ".conv"] = (r, H), (r, c)
            s.update({p + "b": (N, H), p + "A_log": (N,), p + "norm": (V,), p + "a1": (ranks[0], H),
                      p + "a2": (N * D, ranks[0]), p + "dt_bias": (N * D,), p + "g1": (ranks[1], H),
                      p + "g2": (N * V, ranks[1]), p + "o": (H, N * V)})
        else:
            a, b = m["left"], m["right"]
            q, k = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            l, r = p + "left.", p + "right."
            s.update({l + "q": (q, H), l + "k": (k, H), l + "q.norm": (q,), l + "k.norm": (k,),
                      l + "sink": (a["heads"],), l + "g": (q, H), l + "o": (H, q)})
            N, V = b["heads"], b["heads"] * b["vdim"]
            s.update({r + "q": (N * b["dim"], H), r + "k": (N * b["dim"], H), r + "v": (V, H),
                      r + "g": (V, H), r + "o": (H, V), r + "norm": (V,), r + "i": (N, H),
                      r + "i.b": (N,), r + "f": (N, H), r + "f.b": (N,)})
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            s.update({f"l{i}.mlp.gate": (F, H), f"l{i}.mlp.up": (F, H), f"l{i}.mlp.down": (H, F)})
    return s


def random_model(config: dict, seed: int, ranks=(5, 7)) -> dict:
    """Random bf16 weights under which every part has a say: forget gates and decays that reach
    from a few tokens to the whole sequence, sinks of the size of the scores, norm weights and
    biases away from one and zero."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config, ranks).items():
        r = torch.randn(*shape, generator=g)
        if name.endswith(("norm1.b", "norm2.b", "final.norm.b")):
            t = 0.2 * r
        elif name.endswith(("norm", "norm1", "norm2")):
            t = 1.0 + 0.3 * r
        elif name.endswith(".sink"):
            t = 1.0 + r
        elif name.endswith(".f.b"):
            t = 3.0 + 1.5 * r
        elif name.endswith(".i.b"):
            t = 0.5 * r
        elif name.endswith("A_log"):
            t = -1.0 + r
        elif name.endswith("dt_bias"):
            t = -2.0 + r
        elif name.endswith(".conv"):
            t = 0.6 * r
        elif name == "embed":
            t = 0.5 * r
        else:
            t = r * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out
