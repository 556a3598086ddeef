"""Kernels of Vadelix's layers beside the kernels of Fizunex's, Fepopel's and Llama's layers that do the
like, against the measured copy bandwidth and the measured bf16 matrix throughput.

Every launch is timed with CUDA events after a write that flushes L2; median of the iterations.
bytes = what the operation has to read and write once; flops = multiply-adds it needs, times two.
The roofline of a scan counts its state updates at the fp32 rate of the CUDA cores (its states are
fp32).

    python benchmarks/kernels/bench_convolved.py [--prompts 8] [--batch 64] [--width 4096] [--only wkv]
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from bench_recurrent import FP32_TFLOPS, PEAKS, ROOT, place, timeit  # noqa: E402


def cases(lens: list[int], ctx: int, decode: bool, H: int, N: int, G: int, D: int, window: int,
          ff: int, E: int, k: int, F: int, R: int, groups: int):
    """(name, kernel it is compared with or None, callable, bytes, flops, flop rate)."""
    from vllm_gcu_b200.layers.moe import GatedSharedMoE
    from vllm_gcu_b200.ops import cuda as C
    from vllm_gcu_b200.ops._native import call, ptr, stream_ptr
    dev, bf = "cuda", torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, device=dev, generator=g)  # noqa: E731
    T, B = sum(lens), len(lens)
    starts = [ctx - 1] * B if decode else [0] * B
    md = place(lens, starts, decode)
    M, out, peak = T * H, [], PEAKS["bf16_tflops"]

    # residual stream, norms, input convolution
    x, y, yb, lo = rnd(T, H), rnd(T, H).to(bf), rnd(T, H).to(bf), torch.empty(T, H, device=dev, dtype=bf)
    w, wb, taps = torch.ones(H, device=dev), torch.ones(H, device=dev, dtype=bf), 4
    out.append(("add_group_norm", "add + rms_norm", lambda: C.add_group_norm(
        x, y, 0.5, w, groups, 1e-5, lo, out=x), M * 12, 0, 1))
    out.append(("add + rms_norm", None, lambda: C.norm(yb, wb, 1e-5, residual=y), M * 8, 0, 1))
    s, ids = C.moe_topk(rnd(T, E), k, True)
    cap = C.moe_align_cap(T * k, E)
    sid, eid, npp, pos_of = C.moe_align(ids, E, cap)
    ys, sh = rnd(cap, H).to(bf), rnd(T, H).to(bf)
    out.append((f"add_group_norm + {k} expert rows + shared row", "unpermute_sum",
                lambda: C.add_group_norm(x, ys, 0.5, w, groups, 1e-5, lo, out=x, pos_of=pos_of,
                                         row_w=s, shared=sh), M * (12 + 2 * k), 0, 1))
    out.append(("unpermute_sum", None, lambda: call(
        "b200_moe_unpermute_sum", ptr(ys), H, ptr(pos_of), ptr(sh), H, ptr(lo), H, None, T, k, H, 1.0,
        0, stream_ptr()), M * (4 + 2 * k), 0, 1))
    cw, mu = rnd(taps, H), torch.rand(5, H, device=dev, generator=g)
    rings = [rnd(B, n, H).to(bf) for n in (taps - 1, taps)]
    for m, ring in ((None, rings[0]), (mu, rings[1])):
        name = "convolution" + (" + 5 mixtures" if m is not None else "")
        n = 1 if m is None else 5
        rows = torch.empty(n, T, H, device=dev, dtype=bf)
        rows = rows[0] if m is None else rows
        if decode:
            out.append((f"add_group_norm + {name}", "add + rms_norm", lambda m=m, ring=ring, rows=rows:
                        C.add_group_norm(x, y, 0.5, w, groups, 1e-5, lo, out=x, conv=(
                            cw, m, md.positions, md.state_slots, ring, rows, T)),
                        M * (10 + 2 * n + 2 * ring.shape[1] + 2), 0, 1))
        else:
            out.append((name, "token_shift", lambda m=m, ring=ring, rows=rows: C.input_conv(
                y, cw, m, md, ring, rows), M * (2 + 2 * n), 0, 1))
    shift = torch.zeros(H, device=dev)
    out.append(("token_shift", None, lambda: C.token_shift(
        x, shift, bf, None, torch.zeros(B, 1, device=dev, dtype=torch.int32), md.positions,
        md.num_decode_tokens, md.cu_q_prefill, 16), M * 6, 0, 1))

    # time mixing beside the gated delta rule
    wide = rnd(T, 4 * N * D).to(bf)
    r, kk, v, gate = (wide[:, i * N * D:(i + 1) * N * D] for i in range(4))
    z, base, bonus, norm = rnd(T, N * D), torch.full((N * D,), -5.0, device=dev), rnd(N * D), \
        torch.ones(N * D, device=dev)
    inner, w2 = rnd(T, R), rnd(N * D, R).to(bf)
    S = torch.zeros(B, N, D, D, device=dev)
    res = torch.empty(T, N * D, device=dev, dtype=bf)
    stb = B * N * D * D * 4 * (2 if decode else 1)

    def wkv():
        if decode:
            C.wkv_step(r, kk, v, gate, inner, w2, base, bonus, norm, D, D, md.positions,
                       md.state_slots, S, 1e-5, res)
            return
        o = C.wkv(r, kk, v, z, base, bonus, D, D, md, S)
        C.head_norm_gate(o, norm, gate, 1e-5, 1.0, res, act="silu")
    out.append(("wkv (inputs, scan, norm)", "delta (inputs, scan, norm)", wkv,
                T * N * D * (10 + (0 if decode else 4)) + stb, T * N * D * D * 6, FP32_TFLOPS))
    conv = tuple(rnd(4, N * D) for _ in range(3))
    st = {"matrix": S, "taps": torch.zeros(B, 4, 3 * N * D, device=dev, dtype=bf)}
    dtb, alog, nw, bz, wb1 = torch.full((N * D,), -4.0, device=dev), torch.zeros(N, device=dev), \
        torch.ones(D, device=dev), rnd(T, N), rnd(N, H).to(bf)

    def delta():
        if decode:
            C.delta_step(yb, r, kk, v, z, gate, wb1, conv, dtb, alog, nw, D, D, D, md.positions,
                         md.state_slots, st, 1e-5, 1.0, res)
            return
        o = C.delta_rule(r, kk, v, z, bz, conv, dtb, alog, D, D, D, md, st)
        C.head_norm_gate(o, nw, gate, 1e-5, 1.0, res)
    out.append(("delta (inputs, scan, norm)", None, delta, T * N * D * 14 + stb, T * N * D * D * 8,
                FP32_TFLOPS))
    w1, w2f = rnd(R, H).to(bf), rnd(N * D, R).to(bf)
    tb = torch.randn(T, R, device=dev, generator=g).to(bf)
    out.append(("decay, first step (fp32 GEMM)", "fp32 gate GEMM", lambda: C.gemm_bf16(
        yb, w1, epilogue=C.EPI_FP32), (M + w1.numel()) * 2 + T * R * 4, 2 * T * w1.numel(), peak))
    wg = rnd(N, H).to(bf)
    out.append(("fp32 gate GEMM", None, lambda: C.gemm_bf16(yb, wg, epilogue=C.EPI_FP32),
                (M + wg.numel()) * 2 + T * N * 4, 2 * T * wg.numel(), peak))
    if not decode:
        out.append(("decay, second step (fp32 GEMM)", "fp32 decay GEMM", lambda: C.gemm_bf16(
            tb, w2f, epilogue=C.EPI_FP32), (tb.numel() + w2f.numel()) * 2 + T * N * D * 4,
            2 * T * w2f.numel(), peak))
        ta, a2 = rnd(T, 128).to(bf), rnd(N * D, 128).to(bf)
        out.append(("fp32 decay GEMM", None, lambda: C.gemm_bf16(ta, a2, epilogue=C.EPI_FP32),
                    (ta.numel() + a2.numel()) * 2 + T * N * D * 4, 2 * T * a2.numel(), peak))
    mixed, wp = rnd(4, T, H).to(bf), rnd(4 * N * D, H).to(bf)
    proj = torch.empty(T, 4 * N * D, device=dev, dtype=bf)

    tiles4 = torch.arange(4, device=dev, dtype=torch.int32)
    rows4 = torch.tensor([4 * C.GROUP_ROWS], device=dev, dtype=torch.int32)
    padded = rnd(4 * C.GROUP_ROWS, H).to(bf)

    def projections():
        if T <= C.GROUP_ROWS:
            C.gemm_bf16_grouped(padded, wp.view(4, N * D, H), tiles4, rows4)
            return
        for i in range(4):
            at = slice(i * N * D, (i + 1) * N * D)
            C.gemm_bf16(mixed[i], wp[at], out=proj[:, at])
    pf = 2 * T * wp.numel()
    out.append(("four projections", "projection GEMM", projections,
                (4 * M + wp.numel() + T * wp.shape[0]) * 2, pf, peak))
    out.append(("projection GEMM", None, lambda: C.gemm_bf16(yb, wp, out=proj),
                (M + wp.numel() + T * wp.shape[0]) * 2, pf, peak))

    # attention
    bs, per = 16, -(-ctx // 16)
    nb = B * per
    cache, first = (torch.zeros(2, nb, bs, G, D, device=dev, dtype=bf) for _ in range(2))
    cache.normal_(generator=g)
    bt = torch.arange(nb, device=dev, dtype=torch.int32).view(B, per)
    sl = torch.full((B,), ctx, device=dev, dtype=torch.int32)
    slots = torch.cat([bt[i].repeat_interleave(bs)[a:a + n].long() * bs
                       + torch.arange(a, a + n, device=dev) % bs
                       for i, (a, n) in enumerate(zip(starts, lens))])
    qkv = rnd(T, (N + 2 * G) * D).to(bf)
    aq, ak, av = qkv[:, :N * D], qkv[:, N * D:(N + G) * D], qkv[:, (N + G) * D:]
    cs, csf = rnd(ctx + 1, D // 2), rnd(ctx + 1, D)
    qw, kn, share = torch.ones(N * D, device=dev), torch.ones(G * D, device=dev), \
        torch.tensor(0.5, device=dev)
    io = T * (2 * N + 4 * G) * D * 2
    mix = dict(share=share, first=first[1], first_dim=D)
    out.append(("qkv_cache, norms and rotation", "qk_norm_rope_cache", lambda: C.qkv_cache(
        aq, ak, av, qw, kn, 1e-5, cs, md.positions, slots, cache[0], cache[1], D, D, v_norm=True,
        **mix), io + T * G * D * 2, 0, 1))
    out.append(("qkv_cache, temperature", "rope_cache", lambda: C.qkv_cache(
        aq, ak, av, None, None, 1e-5, None, md.positions, slots, cache[0], cache[1], D, D,
        temp=(0.1, 64), **mix), io + T * G * D * 2, 0, 1))
    out.append(("qk_norm_rope_cache", None, lambda: C.qk_norm_rope_cache(
        aq, ak, av, qw, kn, 1e-5, cs, False, md.positions, slots, cache[0], cache[1], D), io, 0, 1))
    out.append(("rope_cache", None, lambda: C.rope_cache_flash(
        aq, ak, av, md.positions, csf, True, D, slots, cache[0], cache[1]), io, 0, 1))
    cache.normal_(generator=g)
    aqc, sink = rnd(T, N, D).to(bf), torch.zeros(N, device=dev)
    slopes = torch.logspace(-8, -0.25, N, base=2.0, device=dev)
    ao = torch.empty_like(aqc)
    tiles = sum(-(-n // 128) for n in lens)

    def att(**kw):
        if decode:
            C.paged_decode(aqc, cache[0], cache[1], bt, sl, 0.09, out=ao,
                           max_seq_len=min(ctx, kw.get("window") or ctx), **kw)
        else:
            kw.setdefault("sink", None)
            C.fmha_prefill_sink(aqc, cache[0], cache[1], bt, md.cu_q_prefill, sl, 0.09, tiles,
                                out=ao, **kw)
    for name, like, win, kw in (
            ("attention with sinks", "attention", ctx, dict(sink=sink)),
            (f"attention, window of {window}, distance bias", "attention", window,
             dict(sink=sink, window=window, slopes=slopes)),
            ("attention, distance bias", "attention", ctx, dict(sink=sink, slopes=slopes)),
            ("attention", None, ctx, {})):
        pairs = sum(min(win, a + i + 1) for a, n in zip(starts, lens) for i in range(n))
        keys = sum(min(a + n, n + win - 1) for a, n in zip(starts, lens))
        out.append((name, like, lambda kw=kw: att(**kw), T * N * D * 4 + keys * G * D * 4,
                    pairs * N * D * 4, peak))

    # feed-forward
    wgu = (rnd(2 * ff, H) * 0.02).to(bf)
    fb, fl = (2 * ff * H + M + T * ff) * 2, 4 * T * ff * H
    out.append(("gate_up + GELU-mul", "gate_up + SiLU-mul", lambda: C.gemm_bf16(
        y, wgu, epilogue=C.EPI_GELU_MUL), fb, fl, peak))
    out.append(("gate_up + SiLU-mul", None, lambda: C.gemm_bf16(
        y, wgu, epilogue=C.EPI_SILU_MUL), fb, fl, peak))
    m = GatedSharedMoE(E, k, 1.0, H, F, F, bf, dev, "x", act="gelu", shared_gate=False)
    for p in m.parameters():
        p.data.normal_(0.0, 0.02)
    touched = int((ids.flatten().bincount(minlength=E) > 0).sum())
    a_s = rnd(cap, H).to(bf)
    for act, like in (("gelu", "grouped up + squared ReLU"), ("relu2", None)):
        name = "grouped up + " + ("GELU" if act == "gelu" else "squared ReLU")
        out.append((name, like, lambda act=act: C.gemm_bf16_grouped(
            a_s, m.experts.w1, eid, npp, act=act), touched * F * H * 2 + T * k * (H + F) * 2,
            2 * T * k * F * H, peak))
    for epi, name, like in ((C.EPI_GELU, "shared up + GELU", "shared up + squared ReLU"),
                            (C.EPI_RELU2, "shared up + squared ReLU", None)):
        out.append((name, like, lambda epi=epi: C.gemm_bf16(
            y, m.shared.up_proj.weight, epilogue=epi), (F * H + M + T * F) * 2, 2 * T * F * H, peak))
    logits = rnd(T, E)
    out.append(("top-k of the best groups", "top-k", lambda: C.moe_topk(logits, k, True, 4, 2),
                T * (E * 4 + k * 8), 0, 1))
    out.append(("top-k", None, lambda: C.moe_topk(logits, k, True), T * (E * 4 + k * 8), 0, 1))
    return out


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__,
                                 formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--prompts", type=int, default=8)
    ap.add_argument("--input-len", type=int, default=1024)
    ap.add_argument("--batch", type=int, default=64)
    ap.add_argument("--width", type=int, default=4096)
    ap.add_argument("--only", default="")
    a = ap.parse_args()
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        PEAKS.update(json.load(open(path)))
    flush = torch.empty(512 << 20, dtype=torch.uint8, device="cuda")
    N = a.width // 128
    sizes = dict(H=a.width, N=N, G=max(1, N // 4), D=128, window=512, ff=7 * a.width // 2, E=32, k=4,
                 F=1536, R=64, groups=8)
    for kind, lens in (("prefill", [a.input_len] * a.prompts), ("decode", [1] * a.batch)):
        for name, like, fn, nbytes, flops, rate in cases(lens, a.input_len, kind == "decode", **sizes):
            if a.only and a.only not in name:
                continue
            ms = timeit(fn, flush)
            roof = max(nbytes / PEAKS["hbm_gbs"] / 1e6, flops / rate / 1e9)
            print(json.dumps({"step": kind, "kernel": name, "us": round(ms * 1e3, 1),
                              "roofline_us": round(roof * 1e3, 1), "frac": round(roof / ms, 3),
                              "like": like}), flush=True)


if __name__ == "__main__":
    main()
