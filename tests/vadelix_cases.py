"""Shared parts of the Vadelix tests: small configurations, weights that make single keys, sinks and
window edges show, and paged batches for kernels.  Engines, schedules and comparisons are those of the
other layer-list families."""
from __future__ import annotations

import torch

import vadelix_oracle as O
from fizunex_cases import Step  # noqa: F401
from sapapel_cases import (errors, mixed_steps, portions, replayer, run, spread,  # noqa: F401
                           tokens_for, write_checkpoint)


def dense(ff) -> dict:
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=0, groups=None) -> dict:
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if groups:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def rotary(heads, kv_heads, dim, vdim, rot, base, scale, yarn=None, mlp=None, mix=True) -> dict:
    """``yarn``: factor, original length, fast, slow."""
    r = {"dims": rot, "base": base}
    if yarn:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                      "rot": r, "v_mix": mix}}


def biased(heads, kv_heads, dim, vdim, window, scale, coef, every, mlp=None, mix=True) -> dict:
    return {"type": "attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                      "mask": {"size": window}, "q_temp": {"coef": coef, "every": every},
                      "v_mix": mix}}


def wkv(heads, dim, mlp=None) -> dict:
    return {"type": "wkv", "mlp": mlp, "mixer": {"heads": heads, "dim": dim}}


def model_config(vocab, width, layers, taps, groups=1, mult=0.6, eps=1e-5) -> dict:
    return {"architecture": "Vadelix", "vocab": vocab, "width": width, "residual_mult": mult,
            "norm": {"eps": eps, "groups": groups}, "canon": {"taps": taps}, "layers": layers}


CONFIGS = {
    # layers of different sizes; the first mixing layer is the second one and has no value norm, later
    # ones split its values into other heads, one does not mix; layers without a feed-forward
    "uneven": model_config(151, 72, [
        wkv(3, 12, moe(6, 3, 24, 20, (3, 2))),
        biased(6, 2, 20, 28, 24, 0.3, 0.4, 7, dense(40)),
        rotary(4, 4, 16, 14, 12, 500.0, 0.31, (3.0, 64, 4.0, 0.25), moe(4, 3, 24)),
        rotary(3, 1, 28, 20, 8, 50.0, 0.2, None, None, False),
        wkv(2, 20)], 4, 3, 0.7, 1e-4),
    # one head of everything, one tap, one group, a window and a temperature step of one, every
    # dimension rotated, one expert
    "ones": model_config(64, 32, [
        rotary(1, 1, 8, 8, 8, 10.0, 1.0, (1.0, 16, 1.0, 1.0), moe(1, 1, 8, 8)),
        wkv(1, 8, dense(1)),
        biased(1, 1, 8, 8, 1, 1.0, 1.0, 1, moe(2, 1, 16, 1, (2, 1)))], 1, 1, 1.0, 1e-6),
    # no size is a multiple of anything, the longest convolution, a rotation without scaling
    "prime": model_config(101, 37, [
        rotary(3, 1, 7, 5, 6, 77.0, 0.6, None, moe(5, 3, 11, 13)),
        wkv(3, 5, dense(23)),
        biased(5, 5, 5, 1, 13, 0.5, 0.7, 11, moe(7, 2, 5)),
        biased(3, 3, 11, 9, 19, 0.4, 0.0, 5, None, False)], 8, 1, 0.5, 1e-4),
    # wider than one tile everywhere, groups of eight heads, a window over several pages and tiles,
    # a norm group for every vector of 8
    "wide": model_config(300, 192, [
        biased(16, 2, 96, 72, 150, 0.12, 0.3, 40, dense(96)),
        rotary(12, 3, 64, 48, 32, 1e5, 0.13, (8.0, 100, 16.0, 0.5), moe(12, 4, 96, 160, (4, 2))),
        wkv(3, 96, moe(8, 2, 64)),
        rotary(8, 2, 128, 72, 128, 1e4, 0.1, (2.0, 1000, 32.0, 1.0), dense(64))], 3, 24, 0.4),
}


def build(folder, name, seed=0, configs=CONFIGS, weights=O.random_model):
    """(configuration, weights, checkpoint folder)"""
    cfg = configs[name]
    w = weights(cfg, seed)
    return cfg, w, write_checkpoint(folder / name, cfg, w)


def peaked_model(config: dict, seed: int) -> dict:
    """Random weights under which single keys, the sinks and far tokens count: attention scores that
    stand out, sinks as large as they, decays near one."""
    w = O.random_model(config, seed)
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}.mix."
        if layer["type"] == "wkv":
            w[p + "w0"] = torch.full_like(w[p + "w0"], -6.0)
            w[p + "w2"] = w[p + "w2"] * 0.1
            continue
        q = p + ("q.norm" if layer["type"] == "attention" else "q")
        w[q] = (w[q].float() * 4.0).to(torch.bfloat16)
        if p + "sink" in w:
            w[p + "sink"] = (w[p + "sink"].float() * 3.0 + 2.0).to(torch.bfloat16)
    return w


def oracle(config: dict, weights: dict, prompts: dict) -> dict:
    return {k: O.forward(config, weights, v) for k, v in prompts.items()}


def greedy(config: dict, weights: dict, prompt, n: int) -> list:
    toks, out = list(prompt), []
    for _ in range(n):
        out.append(int(O.forward(config, weights, toks)[-1].argmax()))
        toks.append(out[-1])
    return out


def clear_choices(config: dict, weights: dict, tokens, gap: float = 0.2) -> torch.Tensor:
    """Rows at which no router's choice is close: the logits of the last chosen group and expert are
    ``gap`` above those of the next ones."""
    real, rows = O.route, torch.ones(len(tokens), dtype=torch.bool)

    def route(h, router, top, groups, keep):
        z = h @ router.T
        T, E = z.shape
        best = z.view(T, groups, -1).max(dim=-1).values.sort(dim=-1, descending=True)
        if keep < groups:
            rows.logical_and_(best.values[:, keep - 1] - best.values[:, keep] > gap)
        open_ = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, best.indices[:, :keep], True)
        s = z.masked_fill(~open_.repeat_interleave(E // groups, dim=1), -1e9)
        s = s.sort(dim=-1, descending=True).values
        if top < E // groups * keep:
            rows.logical_and_(s[:, top - 1] - s[:, top] > gap)
        return real(h, router, top, groups, keep)
    O.route = route
    try:
        O.forward(config, weights, tokens)
    finally:
        O.route = real
    return rows


def windowed_batch(Hq, Hkv, D, q_lens, seq_lens, window, dtype, bs=16, seed=0):
    """Paged keys and values and queries whose keys stand out: a query matches one key it sees (first
    or last of its window, at the edge of a page or tile); the last key in front of its window and the
    first behind the query match better still, so one of them seen by mistake takes over."""
    g = torch.Generator().manual_seed(seed)
    B = len(q_lens)
    mb = max(1, -(-max(seq_lens) // bs)) + 1
    nb = B * mb + 3
    kc, vc = torch.randn(nb, bs, Hkv, D, generator=g), torch.randn(nb, bs, Hkv, D, generator=g)
    bt = (torch.randperm(nb - 1, generator=g)[:B * mb] + 1).view(B, mb).int()
    rows = []
    for b, (ql, n) in enumerate(zip(q_lens, seq_lens)):
        for i in range(ql):
            pos = n - ql + i
            lo = max(0, pos - window + 1) if window else 0
            edges = sorted({c for c in (lo, lo + 1, pos - 1, pos, 0, 1, 15, 16, 63, 64, 127, 128,
                                        255, 256) if lo <= c <= pos})
            for a in range(Hq):
                if not edges:
                    rows.append(torch.randn(D, generator=g))
                    continue

                def key(p, gain):
                    k = kc[bt[b, p // bs], p % bs, a // (Hq // Hkv)]
                    return k * (gain * D ** 0.5 / (k @ k))
                row = key(edges[(a + i) % len(edges)], 8.0)
                if lo > 0:
                    row = row + key(lo - 1, 14.0)
                if pos + 1 < n:
                    row = row + key(pos + 1, 14.0)
                rows.append(row)
    q = torch.stack(rows).view(sum(q_lens), Hq, D)
    cu = torch.tensor([0] + list(torch.tensor(q_lens).cumsum(0)), dtype=torch.int32)
    return (q.to(dtype), kc.to(dtype), vc.to(dtype), bt,
            torch.tensor(seq_lens, dtype=torch.int32), cu)
