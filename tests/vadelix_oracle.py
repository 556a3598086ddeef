"""Plain, slow evaluation of the Vadelix design in torch, one function per mechanism.

Test oracle only: whole sequences, no cache, no batching, nothing shared with the package.  All
functions take and return tensors of the dtype they are given (float32 or float64).

Notation: ``x`` is the residual stream ``[T, H]`` of one sequence, ``h`` a sublayer's input, ``w``
maps tensor names to tensors.  The recurrence is a loop over tokens that holds one matrix per head.
"""
from __future__ import annotations

import math

import torch


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last dimension (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def group_norm(x: torch.Tensor, weight: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """Every one of ``groups`` consecutive parts over its own root mean square; one weight per
    coordinate."""
    parts = [rms_unit(p, eps) for p in x.split(x.shape[-1] // groups, dim=-1)]
    return torch.cat(parts, dim=-1) * weight


def past(x: torch.Tensor, n: int) -> torch.Tensor:
    """The rows of n tokens ago, zeros in front of the sequence."""
    return torch.cat([torch.zeros_like(x[:n]), x[:max(x.shape[0] - n, 0)]])


def input_conv(h: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """``h`` plus a causal convolution of it: ``taps [H, n]``, the last one meets the row itself."""
    n = taps.shape[1]
    return h + sum(taps[:, j] * past(h, n - 1 - j) for j in range(n))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def frequencies(dims: int, base: float, scaling) -> tuple[list[float], float]:
    """Angles per position of the dims / 2 pairs, and the factor of cosines and sines.  Scaled: pairs
    that turn often over the original length keep their frequency, slow ones are divided by the
    factor, a linear ramp over the pair's index lies between."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0

    def pair(turns):           # index of the pair that turns so often over the original length
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(pair(scaling["fast"])), 0)
    hi = min(math.ceil(pair(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        slow = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * slow + fi * (1.0 - slow))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_halves(x: torch.Tensor, dims: int, base: float, scaling=None) -> torch.Tensor:
    """``x [T, heads, dim]`` at positions 0 .. T-1; coordinate i pairs with i + dims / 2, the
    coordinates from ``dims`` on pass."""
    f, gain = frequencies(dims, base, scaling)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    c, s = ((gain * t).to(x.dtype)[:, None] for t in (a.cos(), a.sin()))
    half = dims // 2
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def temperature(T: int, coef: float, every: int) -> torch.Tensor:
    """Factor of the queries at positions 0 .. T-1."""
    return torch.tensor([1.0 + coef * math.log((p + 1) // every + 1) for p in range(T)],
                        dtype=torch.float64)


def slopes(heads: int) -> list[float]:
    return [2.0 ** (-8.0 * (a + 1) / heads) for a in range(heads)]


def visible(T: int, window=None) -> torch.Tensor:
    """[query, key]: keys up to the query, the last ``window`` of them."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < (window or T))


def sink_softmax(scores: torch.Tensor, sink) -> torch.Tensor:
    """Weights over the last dimension with one more term exp(sink) in the denominator."""
    top = torch.clamp(scores.max(dim=-1, keepdim=True).values, min=float(sink))
    e = torch.exp(scores - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def attend(q, k, v, scale: float, sinks, window=None, slope=None) -> torch.Tensor:
    """``q [T, heads, dim]``, ``k, v [T, kv_heads, ...]`` -> ``[T, heads * vdim]``."""
    T, heads = q.shape[:2]
    group = heads // k.shape[1]
    back = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(q.dtype)
    out = []
    for a in range(heads):
        s = q[:, a] @ k[:, a // group].T * scale
        if slope is not None:
            s = s - slope[a] * back
        s = s.masked_fill(~visible(T, window), -math.inf)
        out.append(sink_softmax(s, sinks[a]) @ v[:, a // group])
    return torch.cat(out, dim=-1)


def mix_values(v: torch.Tensor, share, first) -> torch.Tensor:
    """``first``: the flattened values of the first layer that mixes, None in that layer."""
    return v if first is None else (1 - share) * v + share * first.view_as(v)


def rotary_attention(h, w: dict, m: dict, eps: float, first):
    """(output, the layer's values).  ``w``: q, k, v, q.norm, k.norm, sink, vmix, o."""
    T = h.shape[0]
    q = (rms_unit(h @ w["q"].T, eps) * w["q.norm"]).view(T, m["heads"], m["dim"])
    k = (rms_unit(h @ w["k"].T, eps) * w["k.norm"]).view(T, m["kv_heads"], m["dim"])
    rot = m["rot"]
    q, k = (rotate_halves(t, rot["dims"], rot["base"], rot.get("scaling")) for t in (q, k))
    v = rms_unit((h @ w["v"].T).view(T, m["kv_heads"], m["vdim"]), eps)
    if m.get("v_mix"):
        v = mix_values(v, w["vmix"], first)
    return attend(q, k, v, m["scale"], w["sink"]) @ w["o"].T, v


def biased_attention(h, w: dict, m: dict, first):
    """(output, the layer's values).  ``w``: q, k, v, vmix, o."""
    T = h.shape[0]
    q = (h @ w["q"].T).view(T, m["heads"], m["dim"])
    q = q * temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"]).to(h.dtype)[:, None, None]
    k = (h @ w["k"].T).view(T, m["kv_heads"], m["dim"])
    v = (h @ w["v"].T).view(T, m["kv_heads"], m["vdim"])
    if m.get("v_mix"):
        v = mix_values(v, w["vmix"], first)
    zero = torch.zeros(m["heads"], dtype=h.dtype)
    return attend(q, k, v, m["scale"], zero, m["mask"]["size"], slopes(m["heads"])) @ w["o"].T, v


def wkv(r, k, v, decay, bonus) -> torch.Tensor:
    """``r, k, v, decay [T, heads, dim]``, ``bonus [heads, dim]`` -> ``[T, heads, dim]``."""
    T, N, D = k.shape
    out = torch.zeros_like(v)
    S = torch.zeros(N, D, D, dtype=v.dtype)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("nd,ndc->nc", r[t], S + bonus[:, :, None] * kv)
        S = decay[t][:, :, None] * S + kv
    return out


def decays(h, w: dict) -> torch.Tensor:
    return torch.exp(-torch.exp(torch.tanh(h @ w["w1"].T) @ w["w2"].T + w["w0"]))


def wkv_mixer(h, w: dict, m: dict, eps: float) -> torch.Tensor:
    """``w``: mu.r, mu.k, mu.v, mu.g, mu.w, r, k, v, g, w1, w2, w0, u, norm, o."""
    T, N, D = h.shape[0], m["heads"], m["dim"]
    mixed = {c: h + (past(h, 1) - h) * w["mu." + c] for c in "rkvgw"}
    r, k, v = ((mixed[c] @ w[c].T).view(T, N, D) for c in "rkv")
    o = wkv(r, k, v, decays(mixed["w"], w).view(T, N, D), w["u"])
    o = rms_unit(o, eps).reshape(T, N * D) * w["norm"] * silu(mixed["g"] @ w["g"].T)
    return o @ w["o"].T


def dense(h, w: dict) -> torch.Tensor:
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(h, router, top: int, groups: int, keep: int):
    """(expert ids, weights) ``[T, top]``: softmax scores, experts of the ``keep`` groups with the
    largest scores only, weights that sum to one."""
    s = torch.softmax(h @ router.T, dim=-1)
    T, E = s.shape
    best = s.view(T, groups, E // groups).max(dim=-1).values.topk(keep, dim=-1).indices
    open_ = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, best, True)
    open_ = open_.repeat_interleave(E // groups, dim=1)
    ids = s.masked_fill(~open_, -1.0).topk(top, dim=-1).indices
    c = s.gather(1, ids)
    return ids, c / (c.sum(dim=-1, keepdim=True) + 1e-20)


def expert(h, up, down) -> torch.Tensor:
    return gelu_erf(h @ up.T) @ down.T


def experts(h, w: dict, f: dict) -> torch.Tensor:
    r = f["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    ids, c = route(h, w["router"], r["top"], g["count"], g["keep"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        for s in range(r["top"]):
            rows = (ids[:, s] == e).nonzero()[:, 0]
            if len(rows):
                out[rows] += c[rows, s, None] * expert(h[rows], w[f"e{e}.up"], w[f"e{e}.down"])
    if f.get("shared"):
        out = out + expert(h, w["shared.up"], w["shared.down"])
    return out


def sub(w: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def run_layers(config: dict, weights: dict, tokens, dtype=torch.float64) -> list:
    """Residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, groups, gain = config["norm"]["eps"], config["norm"]["groups"], config["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens)]
    out, first = [], None
    for i, layer in enumerate(config["layers"]):
        lw, m = sub(w, f"l{i}."), layer["mixer"]
        mw = sub(lw, "mix.")
        h = input_conv(group_norm(x, lw["norm1"], groups, eps), lw["canon1"])
        if layer["type"] == "wkv":
            y = wkv_mixer(h, mw, m, eps)
        else:
            y, v = rotary_attention(h, mw, m, eps, first) if layer["type"] == "attention" else \
                biased_attention(h, mw, m, first)
            if m.get("v_mix") and first is None:
                first = v.reshape(len(tokens), -1)
        x = x + gain * y
        f = layer["mlp"]
        if f is not None:
            h = group_norm(x, lw["norm2"], groups, eps)
            fw = sub(lw, "mlp.")
            x = x + gain * (dense(h, fw) if f["kind"] == "dense" else experts(h, fw, f))
        out.append(x)
    return out


def forward(config: dict, weights: dict, tokens, dtype=torch.float64) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence."""
    x = run_layers(config, weights, tokens, dtype)[-1]
    n = config["norm"]
    return group_norm(x, weights["final.norm"].to(dtype), n["groups"], n["eps"]) @ \
        weights["head"].to(dtype).T


def tensor_shapes(config: dict, ranks=5) -> dict:
    """Names and shapes of all tensors; ``ranks``: inner width of the decays' two-step projections (no
    number of the configuration)."""
    H = config["width"]
    s = {"embed": (config["vocab"], H), "final.norm": (H,), "head": (config["vocab"], H)}
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        s.update({p + "norm1": (H,), p + "canon1": (H, config["canon"]["taps"])})
        x = p + "mix."
        if layer["type"] == "wkv":
            n = m["heads"] * m["dim"]
            s.update({x + "mu." + c: (H,) for c in "rkvgw"})
            s.update({x + c: (n, H) for c in "rkvg"})
            s.update({x + "w1": (ranks, H), x + "w2": (n, ranks), x + "w0": (n,), x + "norm": (n,),
                      x + "u": (m["heads"], m["dim"]), x + "o": (H, n)})
        else:
            q, k, v = (m[a] * m[b] for a, b in (("heads", "dim"), ("kv_heads", "dim"),
                                                ("kv_heads", "vdim")))
            s.update({x + "q": (q, H), x + "k": (k, H), x + "v": (v, H),
                      x + "o": (H, m["heads"] * m["vdim"])})
            if m.get("v_mix"):
                s[x + "vmix"] = ()
            if layer["type"] == "attention":
                s.update({x + "q.norm": (q,), x + "k.norm": (k,), x + "sink": (m["heads"],)})
        if f is None:
            continue
        s[p + "norm2"] = (H,)
        x = p + "mlp."
        if f["kind"] == "dense":
            s.update({x + "gate": (f["ff"], H), x + "up": (f["ff"], H), x + "down": (H, f["ff"])})
            continue
        s[x + "router"] = (f["router"]["experts"], H)
        names = [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])]
        for n, ff in names + ([("shared", f["shared"]["ff"])] if f.get("shared") else []):
            s.update({f"{x}{n}.up": (ff, H), f"{x}{n}.down": (H, ff)})
    return s


def random_model(config: dict, seed: int, ranks=5) -> dict:
    """Random bf16 weights under which every part has a say: decays that reach from a few tokens to the
    whole sequence, sinks of the size of the scores, mixed values, norm weights away from one, routers
    with clear choices."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config, ranks).items():
        r = torch.randn(*shape, generator=g) if shape else torch.randn((), generator=g)
        if name.endswith(("norm", "norm1", "norm2")):
            t = 1.0 + 0.3 * r
        elif name.endswith(".sink"):
            t = 1.0 + r
        elif name.endswith(".vmix"):
            t = 0.5 + 0.3 * r
        elif name.endswith(".canon1"):
            t = 0.5 * r
        elif ".mu." in name:
            t = torch.rand(*shape, generator=g)
        elif name.endswith(".w0"):
            t = -2.5 + 1.5 * r
        elif name.endswith(".u"):
            t = r
        elif name.endswith(".router"):
            t = 4.0 * r * shape[-1] ** -0.5
        elif name == "embed":
            t = r
        else:
            t = r * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out
