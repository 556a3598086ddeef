"""Plain, slow evaluation of the Sapapel design in torch, one function per mechanism.

Test oracle only: whole sequences, no cache, no batching, nothing shared with the package.  All
functions take and return tensors of the dtype they are given (float32 or float64).

Notation: ``x`` is the residual stream ``[T, H]`` of one sequence, ``w`` maps tensor names to
tensors.
"""
from __future__ import annotations

import math

import torch


def rms_scale(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last dimension (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def scalar_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose gain is one number for all coordinates."""
    return rms_scale(x, eps) * gain.reshape(())


def post_norm(x, y, gain, alpha: float, eps: float):
    """Norm after the weighted residual sum."""
    return scalar_norm(alpha * x + y, gain, eps)


def token_shift(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    """Every row moves towards the row before it, by a fraction per coordinate; the row before
    the first is zero."""
    out = torch.empty_like(h)
    prev = torch.zeros_like(h[0])
    for t in range(h.shape[0]):
        out[t] = h[t] + (prev - h[t]) * mu
        prev = h[t]
    return out


def latent_attention(h: torch.Tensor, w: dict, heads: int, dim: int, vdim: int, scale: float,
                     eps: float) -> torch.Tensor:
    """``w``: q, dkv, dkv.norm, uk, uv, g, o.  Keys and values of every head are expanded from
    the normalised latent rows; causal softmax; sigmoid gate on the concatenated heads."""
    T = h.shape[0]
    q = (h @ w["q"].T).view(T, heads, dim)
    c = rms_scale(h @ w["dkv"].T, eps) * w["dkv.norm"]
    k = (c @ w["uk"].T).view(T, heads, dim)
    v = (c @ w["uv"].T).view(T, heads, vdim)
    out = torch.zeros(T, heads, vdim, dtype=h.dtype)
    for a in range(heads):
        s = (q[:, a] @ k[:, a].T) * scale
        s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], -math.inf)
        e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
        out[:, a] = (e / e.sum(dim=-1, keepdim=True)) @ v[:, a]
    gate = 1.0 / (1.0 + torch.exp(-(h @ w["g"].T)))
    return (out.reshape(T, heads * vdim) * gate) @ w["o"].T


def route(h: torch.Tensor, router: torch.Tensor, top: int):
    """Scores and ids of the ``top`` best experts of every row, not renormalised."""
    s = 1.0 / (1.0 + torch.exp(-(h @ router.T)))
    order = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    return torch.gather(s, 1, order), order


def expert(z: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor):
    g = z @ gate.T
    return ((g / (1.0 + torch.exp(-g))) * (z @ up.T)) @ down.T


def moe(h: torch.Tensor, w: dict, top: int) -> torch.Tensor:
    """``w``: router, e<j>.gate / up / down.  The score scales the expert's input."""
    s, ids = route(h, w["router"], top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for slot in range(top):
            e = int(ids[t, slot])
            out[t] += expert((s[t, slot] * h[t])[None], w[f"e{e}.gate"], w[f"e{e}.up"],
                             w[f"e{e}.down"])[0]
    return out


def depth_average(results: list, weights: torch.Tensor) -> torch.Tensor:
    """Weighted sum of the embedding output and the results of all layers so far."""
    out = torch.zeros_like(results[0])
    for j, r in enumerate(results):
        out = out + weights[j] * r
    return out


def _sub(w: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config: dict, weights: dict, tokens, dtype=torch.float64, want_layers: bool = False):
    """Logits ``[T, vocab]`` of one sequence (and the stream after every layer)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, alpha = float(config["norm"]["eps"]), float(config["postln_alpha"])
    x = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    results, streams = [x], []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        m = layer["mixer"]
        h = token_shift(x, w[p + "shift"])
        y = latent_attention(h, _sub(w, p + "mix."), m["heads"], m["dim"], m["vdim"], m["scale"],
                             eps)
        x = post_norm(x, y, w[p + "norm1"], alpha, eps)
        if layer["mlp"] is not None:
            y = moe(x, _sub(w, p + "mlp."), layer["mlp"]["router"]["top"])
            x = post_norm(x, y, w[p + "norm2"], alpha, eps)
        results.append(x)
        x = depth_average(results, w[p + "dwa"])
        streams.append(x)
    logits = scalar_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, streams) if want_layers else logits


def random_model(config: dict, seed: int = 0, std: float = 1.0, dtype=torch.bfloat16) -> dict:
    """Random weights (rounded to ``dtype``) for a configuration: projections with variance
    ``std^2 / fan_in``, shift fractions in [0, 1), gains around one."""
    g = torch.Generator().manual_seed(seed)
    H, V = config["width"], config["vocab"]

    def mat(o, i):
        return (torch.randn(o, i, generator=g) * std * i ** -0.5).to(dtype)

    def gain():
        return (1.0 + 0.3 * torch.randn((), generator=g)).to(dtype)
    w = {"embed": torch.randn(V, H, generator=g).to(dtype), "head": mat(V, H),
         "final.norm": gain()}
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        A, d, dv, L = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        w.update({p + "norm1": gain(), p + "shift": torch.rand(H, generator=g).to(dtype),
                  p + "mix.q": mat(A * d, H), p + "mix.dkv": mat(L, H),
                  p + "mix.dkv.norm": (1.0 + 0.2 * torch.randn(L, generator=g)).to(dtype),
                  p + "mix.uk": mat(A * d, L), p + "mix.uv": mat(A * dv, L),
                  p + "mix.g": mat(A * dv, H), p + "mix.o": mat(H, A * dv)})
        dwa = 0.3 * torch.randn(i + 2, generator=g)
        dwa[-1] += 1.0
        w[p + "dwa"] = dwa.to(dtype)
        if layer["mlp"] is None:
            continue
        E, F = layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"]
        w.update({p + "norm2": gain(), p + "mlp.router": 2.0 * mat(E, H)})
        for e in range(E):
            w.update({p + f"mlp.e{e}.gate": mat(F, H), p + f"mlp.e{e}.up": mat(F, H),
                      p + f"mlp.e{e}.down": mat(H, F)})
    return w
