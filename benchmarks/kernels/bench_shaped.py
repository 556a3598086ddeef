"""Kernels of Fepopel's layers beside the kernels of DeepSeek's (and Llama's) layers that do the like,
against the measured copy bandwidth and the measured bf16 matrix throughput.

Every launch is timed with CUDA events after a write that flushes L2; median of the iterations.
bytes = what the operation has to read and write once; flops = multiply-adds it needs, times two.

    python benchmarks/kernels/bench_shaped.py [--prompts 8] [--batch 64] [--width 4096] [--only chunk]
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
PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


def timeit(fn, flush, iters: int = 20) -> float:
    for _ in range(3):
        fn()
    ts = []
    for _ in range(iters):
        flush.fill_(1)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    return statistics.median(ts)


def cases(lens: list[int], ctx: int, decode: bool, H: int, N: int, G: int, D: int, L: int, R: int,
          chunk: int, E: int, k: int, F: int):
    """(name, kernel it is compared with or None, callable, bytes, flops)."""
    from vllm_gcu_b200.layers.moe import GatedSharedMoE
    from vllm_gcu_b200.ops import cuda as C
    from vllm_gcu_b200.ops._native import call, ptr, stream_ptr
    dev, bf = "cuda", torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, device=dev, generator=g)  # noqa: E731
    T, B = sum(lens), len(lens)
    starts = [ctx - 1] * B if decode else [0] * B
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lens)]).to(dev)
    cu = None if decode else torch.tensor([0, *lens], device=dev).cumsum(0).int()
    bs, per = 16, -(-ctx // 16)
    nb = B * per
    bt = torch.arange(nb, device=dev, dtype=torch.int32).view(B, per)
    slots = torch.cat([bt[r].repeat_interleave(bs)[s:s + n].long() * bs
                       + torch.arange(s, s + n, device=dev) % bs
                       for r, (s, n) in enumerate(zip(starts, lens))])
    sl = torch.full((B,), ctx, device=dev, dtype=torch.int32)
    out, M = [], T * H

    # residual stream and norms
    x, y, yb = rnd(T, H), rnd(T, H).to(bf), rnd(T, H).to(bf)
    w, wb, lo = torch.ones(H, device=dev), torch.ones(H, device=dev, dtype=bf), torch.empty_like(y)
    out.append(("add_normed + norm", "add + rms_norm", lambda: C.add_normed(
        x, y, w, None, 1e-6, lo, out=x, layer_norm=False, final_weight=w), M * 12, 0))
    out.append(("start_rows + norm", "add + rms_norm", lambda: C.start_rows(
        y, 2.0, weight=w, eps=1e-6), M * 8, 0))
    out.append(("add + rms_norm", None, lambda: C.norm(yb, wb, 1e-6, residual=y), M * 8, 0))
    s, ids = C.moe_topk(rnd(T, E), k, True)
    cap = C.moe_align_cap(T * k, E)
    sid, eid, npp, pos_of = C.moe_align(ids, E, cap)
    ys, sh, gate = rnd(cap, H).to(bf), rnd(T, H).to(bf), rnd(T, 8)
    out.append((f"add_normed + norm + {k} expert rows + gated shared row", "unpermute_sum",
                lambda: C.add_normed(x, ys, w, None, 1e-6, lo, out=x, layer_norm=False,
                                     final_weight=w, pos_of=pos_of, row_w=s, shared=sh,
                                     gate=gate[:, 0]), M * (12 + 2 * k), 0))
    out.append(("unpermute_sum", None, lambda: call(
        "b200_moe_unpermute_sum", ptr(ys), H, ptr(pos_of), ptr(sh), H, ptr(lo), H, None, T, k, H, 1.0,
        0, stream_ptr()), M * (4 + 2 * k), 0))

    # experts
    m = GatedSharedMoE(E, k, 2.0, H, F, F, bf, dev, "x")
    for p in m.parameters():
        p.data.normal_(0.0, 0.02)
    rows = int(npp)
    touched = int((ids.flatten().bincount(minlength=E) > 0).sum())
    a_s, h_s = rnd(cap, H).to(bf), rnd(cap, F).to(bf)
    w13 = (rnd(E, 2 * F, H) * 0.02).to(bf)
    out.append(("grouped up + squared ReLU", "grouped gate_up + SiLU-mul", lambda: C.gemm_bf16_grouped(
        a_s, m.experts.w1, eid, npp, act="relu2"), touched * F * H * 2 + T * k * (H + F) * 2,
        2 * T * k * F * H))
    out.append(("grouped gate_up + SiLU-mul", None, lambda: C.gemm_bf16_grouped(
        a_s, w13, eid, npp, silu_mul=True), touched * F * H * 4 + T * k * (H + F) * 2,
        4 * T * k * F * H))
    out.append(("grouped down", None, lambda: C.gemm_bf16_grouped(h_s, m.experts.w2, eid, npp),
                touched * F * H * 2 + T * k * (H + F) * 2, 2 * T * k * F * H))
    wgu = (rnd(2 * F, H) * 0.02).to(bf)
    out.append(("shared up + squared ReLU", "shared gate_up + SiLU-mul", lambda: C.gemm_bf16(
        y, m.shared.up_proj.weight, epilogue=C.EPI_RELU2), (F * H + M + T * F) * 2, 2 * T * F * H))
    out.append(("shared gate_up + SiLU-mul", None, lambda: C.gemm_bf16(
        y, wgu, epilogue=C.EPI_SILU_MUL), (2 * F * H + M + T * F) * 2, 4 * T * F * H))
    wr, wd = m.router.weight, rnd(E, H).to(bf)
    out.append(("router and shared gate, fp32 GEMM", "router GEMM", lambda: C.gemm_bf16(
        y, wr, epilogue=C.EPI_FP32), (M + wr.numel()) * 2 + T * wr.shape[0] * 4,
        2 * T * wr.numel()))
    out.append(("router GEMM", None, lambda: C.gemm_bf16(y, wd),
                (M + wd.numel()) * 2 + T * wd.shape[0] * 2, 2 * T * wd.numel()))

    # latent attention
    W = -(-(L + R) // 64) * 64
    lc = torch.zeros(nb, bs, W, device=dev, dtype=bf)
    lc.normal_(generator=g)
    q = rnd(T, N * (D + R)).to(bf)
    q_lat, kv, nw, cs = rnd(T, N, W).to(bf), rnd(T, L + R).to(bf), torch.ones(L, device=dev, dtype=bf), \
        rnd(ctx + 1, R)
    io = T * (L + R) * 4 + T * N * R * 4
    out.append(("latent_cache + rotation", "mla_rope_cache", lambda: C.latent_cache(
        kv, nw, 1e-6, lc, slots, cos_sin=cs, positions=pos, q=q, q_lat=q_lat), io, 0))
    out.append(("mla_rope_cache", None, lambda: C.mla_rope_cache(
        q.view(T, N, D + R)[..., D:], kv, pos, cs, nw, 1e-6, lc, slots, L,
        is_neox=False, q_out=q_lat[..., L:L + R]), io, 0))
    sink, lg = rnd(N), rnd(T, N + 8).to(bf)
    o_lat = torch.empty(T, N, L, device=dev, dtype=bf)
    pairs = sum(n * (2 * st + n + 1) // 2 for st, n in zip(starts, lens))
    tiles = sum(-(-n // (128 // N)) for n in lens)

    def mla(**kw):
        C.mla_attention(q_lat, lc, bt, sl, cu, tiles, ctx, W ** -0.5, out=o_lat, L=L, **kw)
    ab, af = T * N * (W + L) * 2 + B * ctx * W * 2, 2 * pairs * N * (W + L)
    out.append(("latent attention, sinks and gates", "latent attention", lambda: mla(
        sink=sink, gate=lg[:, :N]), ab, af))
    out.append(("latent attention", None, mla, ab, af))

    # chunked attention
    qkv = rnd(T, (N + 2 * G) * D).to(bf)
    cq, ck, cv = qkv[:, :N * D], qkv[:, N * D:(N + G) * D], qkv[:, (N + G) * D:]
    cache = torch.zeros(2, nb, bs, G, D, device=dev, dtype=bf)
    cache.normal_(generator=g)
    dw, csf = torch.ones(D, device=dev), rnd(ctx + 1, D)
    io = T * (2 * N + 4 * G) * D * 2
    out.append(("head_norm_cache", "rope_cache", lambda: C.head_norm_cache(
        cq, ck, cv, dw, dw, 1e-6, slots, cache[0], cache[1], D), io, 0))
    out.append(("rope_cache", None, lambda: C.rope_cache_flash(
        cq, ck, cv, pos, csf, True, D, slots, cache[0], cache[1]), io, 0))
    aq, ao = rnd(T, N, D).to(bf), torch.empty(T, N, D, device=dev, dtype=bf)
    t128 = sum(-(-n // 128) for n in lens)

    def seen(c):
        """keys in sight of all queries, keys that are read"""
        pr = rd = 0
        for st, n in zip(starts, lens):
            for p in range(st, st + n):
                pr += p % c + 1 if c else p + 1
            rd += (st + n - 1) % c + 1 if c and n == 1 else n + st
        return pr, rd

    def att(c, cap):
        if decode:
            C.paged_decode(aq, cache[0], cache[1], bt, sl, 0.1, out=ao, max_seq_len=min(ctx, c or ctx),
                           softcap=cap, chunk=c)
        else:
            C.fmha_prefill_sink(aq, cache[0], cache[1], bt, cu, sl, 0.1, t128, None, out=ao,
                                softcap=cap, chunk=c)
    for name, like, c, cap in ((f"attention, chunks of {chunk}, soft cap", "attention", chunk, 50.0),
                               (f"attention, chunks of {chunk}", "attention", chunk, 0.0),
                               ("attention, soft cap", "attention", 0, 50.0),
                               ("attention", None, 0, 0.0)):
        pr, rd = seen(c)
        out.append((name, like, lambda c=c, cap=cap: att(c, cap), T * N * D * 4 + rd * G * D * 4,
                    4 * pr * N * D))
    return out


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__,
                                 formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--prompts", type=int, default=8)
    ap.add_argument("--input-len", type=int, default=1024)
    ap.add_argument("--batch", type=int, default=64)
    ap.add_argument("--width", type=int, default=4096)
    ap.add_argument("--chunk", type=int, default=512)
    ap.add_argument("--experts", type=int, nargs=3, default=[32, 4, 1536],
                    help="experts, experts per token, expert width")
    ap.add_argument("--only", default="")
    a = ap.parse_args()
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        PEAKS.update(json.load(open(path)))
    flush = torch.empty(512 << 20, dtype=torch.uint8, device="cuda")
    sizes = dict(H=a.width, N=a.width // 128, G=max(1, a.width // 512), D=128, L=512, R=64,
                 chunk=a.chunk, **dict(zip("EkF", a.experts)))
    for kind, lens in (("prefill", [a.input_len] * a.prompts), ("decode", [1] * a.batch)):
        rows, fracs = [], {}
        for name, like, fn, nbytes, flops in cases(lens, a.input_len, kind == "decode", **sizes):
            if a.only and a.only not in name:
                continue
            ms = timeit(fn, flush)
            roof = max(nbytes / PEAKS["hbm_gbs"] / 1e6, flops / PEAKS["bf16_tflops"] / 1e9)
            fracs[name] = roof / ms
            rows.append({"step": kind, "kernel": name, "us": round(ms * 1e3, 1),
                         "roofline_us": round(roof * 1e3, 1), "frac": round(roof / ms, 3),
                         "like": like})
        for r in rows:
            if r["like"] in fracs:
                r["like_frac"] = round(fracs[r["like"]], 3)
            print(json.dumps(r), flush=True)


if __name__ == "__main__":
    main()
