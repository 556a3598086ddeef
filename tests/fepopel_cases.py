"""Shared parts of the Fepopel tests: small configurations, weights that make far keys, sinks and
chunk edges show, and paged batches for kernels.  Engines, schedules and comparisons are those of the
other layer-list families."""
from __future__ import annotations

import torch

import fepopel_oracle as O
from sapapel_cases import (errors, mixed_steps, portions, replayer, run, spread,  # noqa: F401
                           tokens_for, write_checkpoint)


def dense(ff) -> dict:
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=0, scale=1.0) -> dict:
    out = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale},
           "expert": {"ff": ff}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def latent(heads, dim, rot, vdim, rank, base, scale, mlp=None) -> dict:
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                      "scale": scale, "rot": {"dims": rot, "base": base}}}


def chunked(heads, kv_heads, dim, vdim, size, scale, softcap, mlp=None) -> dict:
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                      "scale": scale, "softcap": softcap, "mask": {"size": size}}}


def model_config(vocab, width, layers, loop=None, eps=1e-5, embed=3.0) -> dict:
    out = {"architecture": "Fepopel", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "embedding": {"scale": embed}, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CONFIGS = {
    # layers of different sizes; the loop takes the middle, three times; one layer without a
    # feed-forward, one without a shared expert
    "uneven": model_config(151, 72, [
        chunked(6, 3, 20, 28, 24, 0.3, 4.0, dense(40)),
        latent(3, 12, 6, 20, 36, 500.0, 0.31, moe(5, 2, 24, 20, 1.7)),
        latent(5, 16, 10, 8, 40, 20.0, 0.2),
        latent(2, 32, 4, 16, 24, 1e4, 0.4, moe(3, 3, 40))], (1, 3, 3), 1e-4),
    # one head of everything, constants of one, a loop over every layer that runs once
    "ones": model_config(64, 32, [
        latent(1, 8, 2, 8, 8, 10.0, 1.0, moe(1, 1, 8, 8)),
        chunked(1, 1, 8, 8, 16, 1.0, 1.0, moe(2, 1, 16, 1))], (0, 2, 1), 1e-6, 1.0),
    # no size is a multiple of anything, chunks of a prime, no loop, nothing unrotated in a layer
    "prime": model_config(101, 37, [
        latent(3, 5, 2, 7, 9, 77.0, 0.6, moe(5, 3, 11, 13, 0.4)),
        chunked(3, 1, 7, 5, 13, 0.5, 2.5, moe(7, 2, 5)),
        chunked(2, 2, 5, 9, 19, 0.7, 9.0, dense(23))], None, 1e-4),
    # wider than one tile everywhere, groups of eight, chunks over several pages and tiles; the loop
    # ends with the last layer and starts with a chunked one
    "wide": model_config(300, 192, [
        latent(12, 48, 32, 40, 80, 1e6, 0.12, dense(96)),
        chunked(16, 2, 96, 72, 150, 0.12, 20.0, moe(12, 4, 96, 160, 2.0)),
        latent(6, 64, 64, 72, 272, 1e5, 0.1, moe(8, 2, 64, 64))], (1, 3, 2)),
}


def build(folder, name, seed=0, configs=CONFIGS, weights=O.random_model):
    """(configuration, weights, checkpoint folder)"""
    cfg = configs[name]
    w = weights(cfg, seed)
    return cfg, w, write_checkpoint(folder / name, cfg, w)


def peaked_model(config: dict, seed: int) -> dict:
    """Random weights under which single keys and the sinks count: attention scores that stand out,
    sinks as large as they."""
    w = O.random_model(config, seed)
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}.mix."
        q = "q" if layer["type"] == "latent_attention" else "q.norm"
        w[p + q] = (w[p + q].float() * 4.0).to(torch.bfloat16)
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
    """Rows at which no router's choice is close: the last chosen expert's logit is ``gap`` above the
    next one's."""
    real, rows = O.route, torch.ones(len(tokens), dtype=torch.bool)

    def route(h, router, top, scale):
        z = (h @ router.T).sort(dim=-1, descending=True).values
        if top < z.shape[1]:
            rows.logical_and_(z[:, top - 1] - z[:, top] > gap)
        return real(h, router, top, scale)
    O.route = route
    try:
        O.forward(config, weights, tokens)
    finally:
        O.route = real
    return rows


def chunk_edges(n: int, size: int) -> list[int]:
    """Positions just in front of and behind the edges of chunks, pages and tiles below ``n``."""
    at = {0, 1, n - 1}
    for m in (size, 16, 64, 128):
        for e in range(m, n + 1, m):
            at |= {e - 1, e, e + 1}
    return sorted(p for p in at if 0 <= p < n)


def paged_batch(Hq, Hkv, D, q_lens, seq_lens, chunk, dtype, bs=16, seed=0):
    """Paged keys and values and queries whose keys stand out: a query matches one key it sees (at the
    edge of a chunk, page or tile, first or last); the last key in front of its chunk and the first
    behind it match better still, so one of them seen by mistake takes over."""
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
            lo = pos // chunk * chunk if chunk else 0
            edges = [c for c in chunk_edges(max(pos + 1, 1), chunk or 16) if lo <= c <= pos]
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
