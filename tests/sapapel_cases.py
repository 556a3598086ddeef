"""Shared parts of the Sapapel tests: small configurations, engines built from checkpoints written
to a temporary folder, and schedules that are compared with the oracle position by position."""
from __future__ import annotations

import json

import torch

import sapapel_oracle as O


def layer(heads, dim, vdim, rank, scale, experts=0, top=0, ff=0) -> dict:
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}} \
        if experts else None
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale}}


def model_config(vocab, width, alpha, eps, layers) -> dict:
    return {"architecture": "Sapapel", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "postln_alpha": alpha, "layers": layers}


CONFIGS = {
    # layers of different sizes, one without a feed-forward, every expert chosen in the last
    "uneven": model_config(151, 72, 1.7, 1e-4, [layer(3, 20, 28, 36, 0.31, 5, 2, 24),
                                                layer(5, 16, 8, 40, 0.2),
                                                layer(2, 32, 16, 24, 0.4, 3, 3, 40)]),
    # one head, one expert, key and value sizes equal to the latent's
    "ones": model_config(64, 32, 1.0, 1e-6, [layer(1, 32, 32, 32, 0.17, 1, 1, 8),
                                             layer(1, 8, 8, 8, 1.0, 2, 1, 16)]),
    # sizes that are whole tiles nowhere
    "odd": model_config(203, 100, 3.1, 1e-5, [layer(7, 12, 20, 44, 0.25, 9, 4, 20),
                                              layer(3, 28, 12, 52, 0.15, 4, 1, 36)]),
    # no size is a multiple of anything
    "prime": model_config(101, 37, 2.6, 1e-4, [layer(3, 5, 7, 9, 0.6, 5, 3, 11),
                                               layer(1, 3, 11, 13, 0.8, 7, 2, 5)]),
    # wider than one 64-column tile, more heads than a power of two, no feed-forward at the end
    "wide": model_config(500, 192, 2.2, 1e-5, [layer(12, 48, 40, 80, 0.14, 8, 3, 96),
                                               layer(6, 64, 72, 144, 0.12, 12, 2, 64),
                                               layer(20, 16, 16, 272, 0.25)]),
}


def write_checkpoint(folder, config: dict, weights: dict) -> str:
    from vllm_gcu_b200.utils.weights import write_safetensors
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config))
    write_safetensors(str(folder / "model.safetensors"), weights)
    return str(folder)


def tokens_for(config: dict, n: int, seed: int = 0) -> list[int]:
    g = torch.Generator().manual_seed(seed + 100)
    return torch.randint(0, config["vocab"], (n,), generator=g).tolist()


def replayer(path: str, device: str, dtype: str = "float32", max_tokens: int = 1024):
    from vllm_gcu_b200.entrypoints.trace_replay import TraceReplayer, build_engine
    return TraceReplayer(build_engine(path, dtype, max_tokens, device))


def run(rp, prompts: dict, steps: list) -> dict:
    """``steps``: lists of ``(request, count)``; every position's logits are wanted.  A request is
    over with its last token.  Returns ``{request: [tokens, vocab]}``."""
    at = {k: 0 for k in prompts}
    got = {k: [] for k in prompts}
    for st in steps:
        entries, end = [], []
        for rid, n in st:
            lo = at[rid]
            toks = prompts[rid][lo:lo + n]
            assert len(toks) == n
            entries.append({"id": rid, "tokens": toks, "want": list(range(n))})
            at[rid] = lo + n
            if at[rid] == len(prompts[rid]):
                end.append(rid)
        with torch.inference_mode():
            out = rp.step(entries, end)
        k = 0
        for rid, n in st:
            got[rid].append(out[k:k + n])
            k += n
    return {k: torch.cat(v) for k, v in got.items() if v}


def errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Root mean square difference of every position, relative to the spread of the logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.double().std()


def oracle(config: dict, weights: dict, prompts: dict) -> dict:
    return {k: O.forward(config, weights, v) for k, v in prompts.items()}


def portions(n: int, sizes) -> list[int]:
    """``n`` cut into portions of the given sizes, repeated."""
    out, i = [], 0
    while n > 0:
        s = min(n, sizes[i % len(sizes)])
        out.append(s)
        n -= s
        i += 1
    return out


def spread(a: list, b: list) -> list:
    """Steps that run two requests side by side, then what is left of the longer one."""
    steps = [[x, y] for x, y in zip(a, b)]
    rest = a[len(b):] or b[len(a):]
    return steps + [[r] for r in rest]


def mixed_steps(rp_prompts: dict) -> list:
    """Requests of unequal length: portions of some beside single tokens of others, one left out
    of some steps, never more than four live."""
    names = list(rp_prompts)
    left = {k: len(v) for k, v in rp_prompts.items()}
    sizes = {k: [(7, 1, 16, 2, 33)[(i + j) % 5] for j in range(5)] for i, k in enumerate(names)}
    started: list = []
    steps, n = [], 0
    while any(left.values()):
        live = [k for k in started if left[k] > 0]
        for k in names:
            if len(live) < 4 and k not in started:
                started.append(k)
                live.append(k)
        st = []
        for i, k in enumerate(live):
            if len(live) > 1 and (n + i) % 5 == 4:
                continue
            c = min(left[k], sizes[k][n % 5] if left[k] > 12 else 1)
            st.append((k, c))
            left[k] -= c
        steps.append(st)
        n += 1
    return [s for s in steps if s]


def peaked_weights(config: dict, seed: int, sharp: float) -> dict:
    """Random weights whose attention scores stand out: a head then reads one key, near or far, and
    a wrong, missing or extra key changes the logits."""
    w = O.random_model(config, seed)
    for i in range(len(config["layers"])):
        w[f"l{i}.mix.q"] = (w[f"l{i}.mix.q"].float() * sharp).to(torch.bfloat16)
    return w
