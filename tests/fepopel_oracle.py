"""Plain, slow evaluation of the Fepopel design in torch, one function per mechanism.

Test oracle only: whole sequences, no cache, no batching, nothing shared with the package.  All
functions take and return tensors of the dtype they are given (float32 or float64).

Notation: ``x`` is the residual stream ``[T, H]`` of one sequence, ``h`` a sublayer's input, ``w``
maps tensor names to tensors.
"""
from __future__ import annotations

import math

import torch


def rms(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last dimension (eps inside the root), weighted."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def rotate(x: torch.Tensor, base: float) -> torch.Tensor:
    """``x [T, ..., R]``: neighbours (2i, 2i + 1) turned by position * base^(-2i / R)."""
    R = x.shape[-1]
    out = torch.empty_like(x)
    for p in range(x.shape[0]):
        for i in range(R // 2):
            a = p * base ** (-2.0 * i / R)
            u, v = x[p, ..., 2 * i], x[p, ..., 2 * i + 1]
            out[p, ..., 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[p, ..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def softmax_values(s: torch.Tensor, v: torch.Tensor, sink=None) -> torch.Tensor:
    """Scores ``[T, T]`` (-inf: not visible) and values ``[T, D]``; exp(sink) joins the sum."""
    top = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    e = torch.exp(s - top)
    den = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - top)
    return (e / den) @ v


def causal(T: int) -> torch.Tensor:
    i = torch.arange(T)
    return i[None, :] <= i[:, None]


def same_chunk(T: int, size: int) -> torch.Tensor:
    i = torch.arange(T) // size
    return i[None, :] == i[:, None]


def latent_attention(h: torch.Tensor, w: dict, heads: int, dim: int, rot_dim: int, vdim: int,
                     rank: int, scale: float, base: float, eps: float) -> torch.Tensor:
    """``w``: q, dkv, dkv.norm, uk, uv, sink, g, o.  Keys and values of every head are expanded
    from the normalised latent; one rotated key part is shared by all heads; one gate per head."""
    T = h.shape[0]
    q = (h @ w["q"].T).view(T, heads, dim + rot_dim)
    kv = h @ w["dkv"].T
    c = rms(kv[:, :rank], w["dkv.norm"], eps)
    kr = rotate(kv[:, rank:], base)
    qr = rotate(q[..., dim:], base)
    k = (c @ w["uk"].T).view(T, heads, dim)
    v = (c @ w["uv"].T).view(T, heads, vdim)
    gate = sigmoid(h @ w["g"].T)
    out = torch.zeros(T, heads, vdim, dtype=h.dtype)
    for a in range(heads):
        s = (q[:, a, :dim] @ k[:, a].T + qr[:, a] @ kr.T) * scale
        s = s.masked_fill(~causal(T), -math.inf)
        out[:, a] = softmax_values(s, v[:, a], w["sink"][a]) * gate[:, a:a + 1]
    return out.reshape(T, heads * vdim) @ w["o"].T


def chunk_attention(h: torch.Tensor, w: dict, heads: int, kv_heads: int, dim: int, vdim: int,
                    scale: float, softcap: float, size: int, eps: float) -> torch.Tensor:
    """``w``: q, k, v, q.norm, k.norm, o.  Grouped heads, queries and keys normalised per head, soft
    capped scores, keys of the query's own chunk only."""
    T = h.shape[0]
    q = rms((h @ w["q"].T).view(T, heads, dim), w["q.norm"], eps)
    k = rms((h @ w["k"].T).view(T, kv_heads, dim), w["k.norm"], eps)
    v = (h @ w["v"].T).view(T, kv_heads, vdim)
    seen = causal(T) & same_chunk(T, size)
    out = torch.zeros(T, heads, vdim, dtype=h.dtype)
    for a in range(heads):
        b = a // (heads // kv_heads)
        s = softcap * torch.tanh((q[:, a] @ k[:, b].T) * scale / softcap)
        out[:, a] = softmax_values(s.masked_fill(~seen, -math.inf), v[:, b])
    return out.reshape(T, heads * vdim) @ w["o"].T


def dense(h: torch.Tensor, w: dict) -> torch.Tensor:
    g = h @ w["gate"].T
    return (g * sigmoid(g) * (h @ w["up"].T)) @ w["down"].T


def expert(h: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    u = torch.clamp(h @ up.T, min=0.0)
    return (u * u) @ down.T


def route(h: torch.Tensor, router: torch.Tensor, top: int, scale: float):
    """Weights and ids of the ``top`` best experts of every row."""
    z = h @ router.T
    e = torch.exp(z - z.max(dim=-1, keepdim=True).values)
    s = e / e.sum(dim=-1, keepdim=True)
    order = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    best = torch.gather(s, 1, order)
    return best / (best.sum(dim=-1, keepdim=True) + 1e-20) * scale, order


def moe(h: torch.Tensor, w: dict, top: int, scale: float) -> torch.Tensor:
    """``w``: router, e<j>.up / down and with a shared expert shared.up / down / sg."""
    s, ids = route(h, w["router"], top, scale)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for slot in range(top):
            e = int(ids[t, slot])
            out[t] += s[t, slot] * expert(h[t:t + 1], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    if "shared.up" in w:
        out = out + sigmoid(h @ w["shared.sg"].T) * expert(h, w["shared.up"], w["shared.down"])
    return out


def below(w: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def mixer(h: torch.Tensor, w: dict, layer: dict, eps: float) -> torch.Tensor:
    m = layer["mixer"]
    if layer["type"] == "latent_attention":
        return latent_attention(h, w, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"],
                                m["scale"], m["rot"]["base"], eps)
    return chunk_attention(h, w, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"],
                           m["softcap"], m["mask"]["size"], eps)


def feed_forward(h: torch.Tensor, w: dict, mlp: dict) -> torch.Tensor:
    if mlp["kind"] == "dense":
        return dense(h, w)
    return moe(h, w, mlp["router"]["top"], mlp["router"]["scale"])


def layer_runs(config: dict) -> list:
    """``(layer, pass or None)`` in the order in which they run; the pass number stands at the first
    layer of every pass of the loop."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(config: dict, weights: dict, tokens, dtype=torch.float64, trace: list | None = None
            ) -> torch.Tensor:
    """Logits ``[T, vocab]``; ``trace`` takes the residual stream after every layer run."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * config["embedding"]["scale"]
    for i, t in layer_runs(config):
        layer, p = config["layers"][i], f"l{i}."
        if t is not None:
            x = x + w["loop.step"][t]
        y = mixer(rms(x, w[p + "norm1"], eps), below(w, p + "mix."), layer, eps)
        x = x + rms(y, w[p + "norm1b"], eps)
        if layer.get("mlp"):
            y = feed_forward(rms(x, w[p + "norm2"], eps), below(w, p + "mlp."), layer["mlp"])
            x = x + rms(y, w[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x)
    return rms(x, w["final.norm"], eps) @ w["head"].T


def random_model(config: dict, seed: int = 0) -> dict:
    """bfloat16 tensors under the names and shapes of a checkpoint."""
    g = torch.Generator().manual_seed(seed)

    def mat(n, m, gain=1.0):
        return (torch.randn(n, m, generator=g) * gain * m ** -0.5).to(torch.bfloat16)

    def near_one(*shape):
        return (1.0 + 0.2 * torch.randn(*shape, generator=g)).to(torch.bfloat16)
    H, V = config["width"], config["vocab"]
    w = {"embed": (torch.randn(V, H, generator=g) * 0.3).to(torch.bfloat16), "head": mat(V, H),
         "final.norm": near_one(H)}
    if config.get("loop"):
        w["loop.step"] = (0.3 * torch.randn(config["loop"]["times"], H, generator=g)).to(torch.bfloat16)
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        A, D, E = m["heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            w[p + n] = near_one(H)
        if layer["type"] == "latent_attention":
            R, L = m["rot_dim"], m["kv_rank"]
            w.update({p + "mix.q": mat(A * (D + R), H, 1.5), p + "mix.dkv": mat(L + R, H),
                      p + "mix.dkv.norm": near_one(L), p + "mix.uk": mat(A * D, L),
                      p + "mix.uv": mat(A * E, L), p + "mix.g": mat(A, H),
                      p + "mix.sink": torch.randn(A, generator=g).to(torch.bfloat16)})
        else:
            G = m["kv_heads"]
            w.update({p + "mix.q": mat(A * D, H), p + "mix.k": mat(G * D, H),
                      p + "mix.v": mat(G * E, H), p + "mix.q.norm": near_one(D),
                      p + "mix.k.norm": near_one(D)})
        w[p + "mix.o"] = mat(H, A * E)
        if f and f["kind"] == "dense":
            w.update({p + "mlp.gate": mat(f["ff"], H), p + "mlp.up": mat(f["ff"], H),
                      p + "mlp.down": mat(H, f["ff"])})
        elif f:
            w[p + "mlp.router"] = mat(f["router"]["experts"], H, 2.0)
            for e in range(f["router"]["experts"]):
                w[f"{p}mlp.e{e}.up"] = mat(f["expert"]["ff"], H)
                w[f"{p}mlp.e{e}.down"] = mat(H, f["expert"]["ff"])
            if f.get("shared"):
                w.update({p + "mlp.shared.up": mat(f["shared"]["ff"], H),
                          p + "mlp.shared.down": mat(H, f["shared"]["ff"]),
                          p + "mlp.shared.sg": mat(1, H)})
    return w
