"""Shared parts of the Fizunex tests: small configurations and weights that make far tokens show.
Engines, schedules and comparisons are those of the other layer-list family."""
from __future__ import annotations

import torch

import fizunex_oracle as O
from sapapel_cases import (errors, mixed_steps, portions, replayer, run, spread,  # noqa: F401
                           tokens_for, write_checkpoint)


def delta(heads, kv_heads, dim, vdim, conv, ff=0) -> dict:
    return {"type": "channel_delta", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def parallel(left, right, scales=(0.8, 1.3), ff=0) -> dict:
    """``left``: heads, kv_heads, dim, rotated dims, base, scale; ``right``: heads, dim, vdim, cap."""
    h, g, d, rot, base, scale = left
    n, rd, rv, cap = right
    return {"type": "parallel", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"left": {"heads": h, "kv_heads": g, "dim": d, "vdim": d, "scale": scale,
                               "rot": {"dims": rot, "base": base}},
                      "right": {"heads": n, "dim": rd, "vdim": rv, "gate_cap": cap},
                      "left_scale": scales[0], "right_scale": scales[1]}}


def model_config(vocab, width, layers, eps=1e-5, embed=1.7, logits=0.6) -> dict:
    return {"architecture": "Fizunex", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embed}, "logit_scale": logits, "layers": layers}


CONFIGS = {
    # layers of different sizes, grouped heads, with and without a feed-forward
    "uneven": model_config(151, 72, [delta(6, 3, 20, 28, 3, 24),
                                     parallel((6, 2, 20, 12, 1000.0, 0.3), (3, 12, 20, 9.0), ff=40),
                                     delta(2, 2, 16, 12, 2),
                                     parallel((4, 4, 16, 16, 50.0, 0.2), (2, 8, 24, 5.0))], 1e-4),
    # one head of everything, a convolution of one tap, all dimensions rotated, constants of one
    "ones": model_config(64, 32, [parallel((1, 1, 8, 8, 10.0, 1.0), (1, 8, 8, 1.0), (1.0, 1.0), 8),
                                  delta(1, 1, 8, 8, 1, 16)], 1e-6, 1.0, 1.0),
    # no size is a multiple of anything, no rotation
    "prime": model_config(101, 37, [delta(3, 1, 5, 7, 5, 11),
                                    parallel((3, 3, 7, 4, 77.0, 0.5), (2, 3, 11, 4.0), ff=13),
                                    parallel((2, 1, 6, 0, 10.0, 0.4), (1, 5, 3, 6.0))], 1e-4),
    # heads wider than one pass of a warp, values wider than keys and the other way round
    "wide": model_config(300, 192, [delta(4, 2, 96, 160, 4, 64),
                                    parallel((8, 4, 96, 32, 1e4, 0.1), (2, 160, 48, 12.0), ff=96),
                                    delta(2, 1, 136, 40, 7)]),
}


def build(folder, name, seed=0, configs=CONFIGS, far=None):
    """(configuration, weights, checkpoint folder).  ``far``: see :func:`far_weights`."""
    cfg = configs[name]
    w = O.random_model(cfg, seed) if far is None else far_weights(cfg, seed, far)
    return cfg, w, write_checkpoint(folder / name, cfg, w)


def far_weights(config: dict, seed: int, sharp: float) -> dict:
    """Random weights under which far tokens count: attention heads that read few keys (their
    norm weights scaled), forget gates and decays near one."""
    w = O.random_model(config, seed)
    for k in w:
        if k.endswith("left.q.norm"):
            w[k] = (w[k].float() * sharp).to(torch.bfloat16)
        elif k.endswith("A_log"):
            w[k] = torch.full_like(w[k], -5.0)
        elif k.endswith("right.f.b"):
            w[k] = torch.full_like(w[k], 30.0)
    return w


def oracle(config: dict, weights: dict, prompts: dict) -> dict:
    return {k: O.forward(config, weights, v) for k, v in prompts.items()}


def greedy(config: dict, weights: dict, prompt, n: int) -> list:
    toks, out = list(prompt), []
    for _ in range(n):
        out.append(int(O.forward(config, weights, toks)[-1].argmax()))
        toks.append(out[-1])
    return out


class Step:
    """One step of several requests as kernels and layers see it: ``(slot, start, count)`` per
    request, single tokens first; ``pad`` rows behind the last request."""

    def __init__(self, requests, pad=0, device="cpu", decodes=None):
        self.requests = requests
        nd = sum(1 for _, _, n in requests if n == 1) if decodes is None else decodes
        assert all(n == 1 for _, _, n in requests[:nd])
        pos = [torch.arange(s, s + n) for _, s, n in requests] + [torch.zeros(pad)]
        counts = [n for _, _, n in requests]
        self.T = sum(counts) + pad
        self.positions = torch.cat(pos).long().to(device)
        self.state_slots = torch.tensor([r[0] for r in requests], dtype=torch.int32, device=device)
        self.num_decode_tokens = nd
        self.cu_q_prefill = torch.tensor([0, *counts[nd:]]).cumsum(0).int().to(device) \
            if counts[nd:] else None
        self.spans, at = [], 0
        for n in counts:
            self.spans.append((at, at + n))
            at += n
        self.is_dummy = False

    def to(self, device):
        out = Step.__new__(Step)
        out.__dict__.update({k: v.to(device) if torch.is_tensor(v) else v
                             for k, v in self.__dict__.items()})
        return out
