"""Kernels of the fp32 residual stream and of the latent cache (Sapapel) beside the kernels of
DeepSeek's layers that do the like, against the measured copy bandwidth.

Every launch is timed with CUDA events after a write that flushes L2; median of the iterations.
bytes = what the operation has to read and write once.

    python benchmarks/kernels/bench_residual.py [--tokens 8192 64] [--width 4096]
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
sys.path.insert(0, ROOT)


def timeit(fn, flush, iters: int = 20) -> float:
    for _ in range(3):
        fn()
    ts = []
    for _ in range(iters):
        flush.fill_(1.0)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    return statistics.median(ts)


def cases(T: int, H: int, L: int = 512, D: int = 4096, k: int = 4, E: int = 32, n: int = 8):
    """(name, like kernel or None, callable, bytes)."""
    from vllm_gcu_b200.ops import cuda as C
    from vllm_gcu_b200.ops._native import call, ptr, stream_ptr
    dev, bf = "cuda", torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, device=dev, generator=g)  # noqa: E731
    x, mu = rnd(T, H), torch.rand(H, device=dev, generator=g)
    xb, rb, wb = rnd(T, H).to(bf), rnd(T, H).to(bf), torch.ones(H, device=dev, dtype=bf)
    hist, w = rnd(n + 1, T, H), rnd(n + 1)
    one = torch.ones((), device=dev)
    res, avg, lo = torch.empty_like(x), torch.empty_like(x), torch.empty_like(xb)
    s, ids = C.moe_topk(rnd(T, E), k, False, sigmoid=True)
    cap = C.moe_align_cap(T * k, E)
    sid, eid, npp, pos = C.moe_align(ids, E, cap)
    ys, yo = rnd(cap, H).to(bf), torch.empty(cap, H, device=dev, dtype=bf)
    bs, nb = 16, -(-T // 16) + 1
    pos_t = torch.arange(T, device=dev)
    bt = torch.arange(nb, device=dev, dtype=torch.int32).view(1, nb)
    cu = torch.tensor([0, T], device=dev, dtype=torch.int32)
    st, cache = rnd(nb, H), torch.zeros(nb, bs, L, device=dev, dtype=bf)
    cache_d = torch.zeros(nb, bs, L + 64, device=dev, dtype=bf)
    kv, kvd = rnd(T, L).to(bf), rnd(T, L + 64).to(bf)
    cs = rnd(T, 64)
    nw = torch.ones(L, device=dev, dtype=bf)
    o, z = rnd(T, D).to(bf), rnd(T, D).to(bf)
    gu = rnd(T, 2 * D).to(bf)
    M = T * H
    rows = int(npp)

    def permute_weighted():
        call("b200_moe_permute_weighted", ptr(x), H, ptr(s), ptr(yo), H, ptr(sid), ptr(npp), T * k,
             k, H, H, cap, 0, stream_ptr())

    def permute():
        call("b200_moe_permute", ptr(xb), H, ptr(yo), H, ptr(sid), ptr(npp), T * k, k, H, cap, 0,
             stream_ptr())

    def unpermute():
        call("b200_moe_unpermute_sum", ptr(ys), H, ptr(pos), None, 0, ptr(lo), H, None, T, k, H,
             1.0, 0, stream_ptr())
    norm = lambda: C.norm(xb, wb, 1e-6, residual=rb)  # noqa: E731
    return [
        ("token_shift", lambda: C.token_shift(x, mu, bf, st, bt, pos_t, 0, cu, bs), M * 6),
        ("post_norm", lambda: C.post_norm(x, xb, one, 2.0, 1e-6, res=res, lo=lo), M * 12),
        (f"post_norm + {k} expert rows + average of {n}",
         lambda: C.post_norm(x, ys, one, 2.0, 1e-6, pos_of=pos, k=k, res=hist[n], hist=hist, n=n,
                             weights=w, avg=avg), M * (12 + 2 * k + 4 * n)),
        ("  like: add + rms_norm", norm, M * 8),
        ("  like: unpermute_sum", unpermute, M * (2 * k + 2)),
        ("permute_weighted", permute_weighted, M * 4 + rows * H * 2),
        ("  like: permute", permute, M * 2 + rows * H * 2),
        ("latent_cache + state", lambda: C.latent_cache(kv, nw, 1e-6, cache, pos_t, x, st, 0, cu),
         T * L * 4 + T // bs * H * 8),
        ("  like: mla_rope_cache", lambda: C.mla_rope_cache(None, kvd, pos_t, cs, nw, 1e-6, cache_d,
                                                           pos_t, L), T * (L + 64) * 4 + T * 256),
        ("sigmoid_gate", lambda: C.sigmoid_gate(o, z), T * D * 6),
        ("  like: silu_mul", lambda: C.activation(gu, "silu"), T * D * 6),
    ]


def attention_cases(T: int, N: int, ctx: int, flush):
    """Latent attention by latent width: prefill of whole prompts and decode, next to the 512 + 64
    wide layout of DeepSeek."""
    from vllm_gcu_b200.ops import cuda as C
    dev = "cuda"
    for L, W in ((128, 128), (256, 256), (384, 384), (512, 512), (512, 576)):
        for decode in (False, True):
            B = min(T, 256) if decode else max(1, T // ctx)
            ql = 1 if decode else ctx
            mb = -(-ctx // 16)
            cache = (torch.randn(B * mb, 16, W, device=dev) * 0.3).to(torch.bfloat16)
            bt = torch.arange(B * mb, device=dev, dtype=torch.int32).view(B, mb)
            sl = torch.full((B,), ctx, device=dev, dtype=torch.int32)
            cu = torch.arange(0, (B + 1) * ql, ql, device=dev, dtype=torch.int32)
            q = (torch.randn(B * ql, N, W, device=dev) * 0.3).to(torch.bfloat16)
            tiles = B * -(-ql // (128 // N))
            t = timeit(lambda: C.mla_attention(q, cache, bt, sl, None if decode else cu, tiles,
                                               ctx, W ** -0.5, L=L), flush)
            pairs = B * N * (ctx if decode else ctx * (ctx + 1) // 2)
            tf = 2.0 * pairs * (W + L) / (t * 1e-3) / 1e12
            gb = B * ctx * W * 2 / (t * 1e-3) / 1e9
            yield {"attention": "decode" if decode else "prefill", "L": L, "W": W, "heads": N,
                   "requests": B, "ctx": ctx, "us": round(t * 1e3, 1), "tflops": round(tf, 1),
                   "cache_gb_s": round(gb, 1)}


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__,
                                 formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--tokens", type=int, nargs="*", default=[8192, 64])
    ap.add_argument("--width", type=int, default=4096)
    ap.add_argument("--heads", type=int, default=32)
    ap.add_argument("--ctx", type=int, default=1024)
    a = ap.parse_args()
    try:
        peak = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json")))["hbm_gbs"]
    except OSError:
        peak = 6650.0
    flush = torch.empty(64 << 20, device="cuda")        # 256 MB, larger than L2
    for T in a.tokens:
        print(f"# {T} tokens, width {a.width}; peak {peak:.0f} GB/s (measured copy)")
        for name, fn, nbytes in cases(T, a.width, D=a.heads * 128):
            t = timeit(fn, flush)
            gbs = nbytes / (t * 1e-3) / 1e9
            print(f"{name:44s} {t * 1e3:8.1f} us {nbytes / 1e6:8.1f} MB {gbs:7.0f} GB/s "
                  f"{gbs / peak:5.2f}", flush=True)
        for line in attention_cases(T, a.heads, a.ctx, flush):
            print(json.dumps(line), flush=True)


if __name__ == "__main__":
    main()
