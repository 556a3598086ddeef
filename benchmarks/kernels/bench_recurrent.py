"""Kernels of Fizunex's layers beside the kernels of Llama's layers that do the like, against the
measured copy bandwidth and the measured bf16 matrix throughput.

Every launch is timed with CUDA events after a write that flushes L2; median of the iterations.
bytes = what the operation has to read and write once; flops = multiply-adds it needs, times two.
The roofline of a scan counts its state updates at the fp32 rate of the CUDA cores (its states are
fp32), the attention kernels' at the measured bf16 rate.

    python benchmarks/kernels/bench_recurrent.py [--tokens 8192] [--batch 64] [--only scan]
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import sys
import types

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
sys.path.insert(0, ROOT)
FP32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12      # CUDA cores at the highest clock


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


def place(lens: list[int], starts: list[int], decode: bool):
    """Positions, portions and state slots of a step, as the kernels take them."""
    dev = "cuda"
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lens)]).to(dev)
    nd = len(lens) if decode else 0
    cu = None if decode else torch.tensor([0, *lens], device=dev).cumsum(0).int()
    return types.SimpleNamespace(positions=pos, num_decode_tokens=nd, cu_q_prefill=cu,
                                 state_slots=torch.arange(len(lens), device=dev).int())


def cases(lens: list[int], ctx: int, decode: bool, H: int, N: int, G: int, D: int, MN: int,
          MD: int, MV: int, ff: int):
    """(name, kernel it is compared with or None, callable, bytes, flops, flop rate)."""
    from vllm_gcu_b200.ops import cuda as C
    dev, bf = "cuda", torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, device=dev, generator=g)  # noqa: E731
    T, B = sum(lens), len(lens)
    starts = [ctx - 1] * B if decode else [0] * B
    md = place(lens, starts, decode)
    ntaps, out = 4, []
    # residual stream
    x, y = rnd(T, H), rnd(T, H).to(bf)
    w, b = torch.ones(H, device=dev), torch.zeros(H, device=dev)
    lo, xb, wb = torch.empty_like(y), rnd(T, H).to(bf), torch.ones(H, device=dev, dtype=bf)
    out.append(("add_normed", "norm", lambda: C.add_normed(x, y, w, b, 1e-5, lo, out=x),
                T * H * 12, 0, 1))
    out.append(("norm", None, lambda: C.norm(xb, wb, 1e-5, residual=y), T * H * 8, 0, 1))
    # gated delta rule
    wide = rnd(T, 3 * N * D + 256).to(bf)
    q, k, v = (wide[:, i * N * D:(i + 1) * N * D] for i in range(3))
    z, bz = rnd(T, N * D), rnd(T, N)
    conv = tuple(rnd(ntaps, N * D) for _ in range(3))
    st = {"matrix": torch.zeros(B, N, D, D, device=dev),
          "taps": torch.zeros(B, ntaps, 3 * N * D, device=dev, dtype=bf)}
    dtb, alog = torch.full((N * D,), -4.0, device=dev), torch.zeros(N, device=dev)
    io = T * N * D * (3 * 2 + 4 + 2)             # projections in, decays in, result out
    stb = B * N * D * D * 4 * (2 if decode else 1)
    gate, nw = rnd(T, N * D).to(bf), torch.ones(D, device=dev)
    res = torch.empty(T, N * D, device=dev, dtype=bf)

    wb1 = rnd(N, H).to(bf)

    def delta():
        if decode:
            C.delta_step(xb, q, k, v, z, gate, wb1, conv, dtb, alog, nw, D, D, D, md.positions,
                         md.state_slots, st, 1e-5, 1.0, res)
            return
        o = C.delta_rule(q, k, v, z, bz, conv, dtb, alog, D, D, D, md, st)
        C.head_norm_gate(o, nw, gate, 1e-5, 1.0, res)
    out.append(("delta (inputs, scan, norm)", "attention", delta, io + stb, T * N * D * D * 8,
                FP32_TFLOPS))
    # matrix memory
    mw = rnd(T, MN * (2 * MD + 2 * MV)).to(bf)
    mq, mk, mv, mg = mw.split([MN * MD, MN * MD, MN * MV, MN * MV], dim=1)
    zi, zf = (rnd(T, 2 * MN)[:, i * MN:(i + 1) * MN] for i in range(2))
    ms = {"matrix": torch.zeros(B, MN, MV, MD, device=dev),
          "vector": torch.zeros(B, MN, MD, device=dev), "scalar": torch.zeros(B, MN, device=dev)}
    ib, fb = torch.zeros(MN, device=dev), torch.full((MN,), 5.0, device=dev)
    mnw = torch.ones(MN * MV, device=dev)
    mres = torch.empty(T, MN * MV, device=dev, dtype=bf)

    wi, wf = rnd(MN, H).to(bf), rnd(MN, H).to(bf)

    def memory():
        if decode:
            C.memory_step(xb, mq, mk, mv, mg, wi, wf, ib, fb, 15.0, mnw, MD, MV, MD, md.positions,
                          md.state_slots, ms, 1e-5, 1.0, mres)
            return
        o, nq, low = C.matrix_memory(mq, mk, mv, zi, zf, ib, fb, 15.0, MD, MV, MD, md, ms)
        C.head_norm_gate(o, mnw, mg, 1e-5, 1.0, mres, nq, low)
    out.append(("memory (inputs, scan, norm)", "attention", memory,
                T * MN * (2 * MD + 3 * MV) * 2 + B * MN * MD * MV * 4 * (2 if decode else 1),
                T * MN * MD * MV * 6, FP32_TFLOPS))
    # attention
    bs = 16
    per = -(-ctx // bs)
    nb = B * per
    cache = torch.zeros(2, nb, bs, G, D, device=dev, dtype=bf)
    cache.normal_(generator=g)
    bt = torch.arange(nb, device=dev, dtype=torch.int32).view(B, per)
    sl = torch.full((B,), ctx, device=dev, dtype=torch.int32)
    qkv = rnd(T, (2 * N + 2 * G) * D).to(bf)
    aq, ak, ag = qkv[:, :N * D], qkv[:, N * D:(N + G) * D], qkv[:, (N + G) * D:(2 * N + G) * D]
    av = qkv[:, (2 * N + G) * D:]
    slots = torch.cat([bt[r].repeat_interleave(bs)[s:s + n].long() * bs
                       + torch.arange(s, s + n, device=dev) % bs
                       for r, (s, n) in enumerate(zip(starts, lens))])
    cs = rnd(ctx + 1, D // 2)
    cs_full = rnd(ctx + 1, D)
    qw, kw, sink = torch.ones(N * D, device=dev), torch.ones(G * D, device=dev), rnd(N)
    out.append(("qk_norm_rope_cache", "rope_cache", lambda: C.qk_norm_rope_cache(
        aq, ak, None, qw, kw, 1e-5, cs, False, md.positions, slots, cache[0], cache[1], D),
        T * (2 * N + 3 * G) * D * 2, 0, 1))
    out.append(("rope_cache", None, lambda: C.rope_cache_flash(
        aq, ak, av, md.positions, cs_full, True, D, slots, cache[0], cache[1]),
        T * (2 * N + 4 * G) * D * 2, 0, 1))
    aqc = rnd(T, N, D).to(bf)
    ao = torch.empty_like(aqc)
    tiles = sum(-(-n // 128) for n in lens)
    pairs = sum(n * (2 * s + n + 1) // 2 for s, n in zip(starts, lens))
    peak = PEAKS["bf16_tflops"]
    abytes = T * N * D * 4 + B * ctx * G * D * 4
    if decode:
        att = lambda s: C.paged_decode(aqc, cache[0], cache[1], bt, sl, 0.1, out=ao,  # noqa: E731
                                       max_seq_len=ctx, sink=s)
    else:
        att = lambda s: C.fmha_prefill_sink(aqc, cache[0], cache[1], bt, md.cu_q_prefill,  # noqa: E731
                                            sl, 0.1, tiles, s, out=ao)
    out.append(("attention with sinks", "attention", lambda: att(sink), abytes, pairs * N * D * 4,
                peak))
    out.append(("attention", None, lambda: att(None), abytes, pairs * N * D * 4, peak))
    hres = torch.empty(T, N * D, device=dev, dtype=bf)
    out.append(("head_gate", "silu_mul", lambda: C.head_gate(ao, ag, 0.7, D, hres), T * N * D * 6, 0,
                1))
    gu = rnd(T, 2 * N * D).to(bf)
    out.append(("silu_mul", None, lambda: C.activation(gu, "silu"), T * N * D * 6, 0, 1))
    # gates with fp32 results beside the GEMM of the projections
    wg = rnd(max(8, N), H).to(bf)
    out.append(("fp32 gate GEMM", "projection GEMM", lambda: C.gemm_bf16(
        xb, wg, epilogue=C.EPI_FP32), (T * H + wg.numel()) * 2 + T * wg.shape[0] * 4,
        2 * T * wg.numel(), peak))
    wp = rnd(3 * N * D, H).to(bf)
    out.append(("projection GEMM", None, lambda: C.gemm_bf16(xb, wp),
                (T * H + wp.numel() + T * wp.shape[0]) * 2, 2 * T * wp.numel(), peak))
    return out


PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


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
    sizes = dict(H=a.width, N=N, G=max(1, N // 4), D=128, MN=N // 4, MD=128, MV=256,
                 ff=7 * a.width // 2)
    for kind, lens in (("prefill", [a.input_len] * a.prompts), ("decode", [1] * a.batch)):
        rows = {}
        for name, like, fn, nbytes, flops, rate in cases(lens, a.input_len, kind == "decode",
                                                         **sizes):
            if a.only and a.only not in name:
                continue
            ms = timeit(fn, flush)
            roof = max(nbytes / PEAKS["hbm_gbs"] / 1e6, flops / rate / 1e9)
            rows[name] = roof / ms
            print(json.dumps({"step": kind, "kernel": name, "us": round(ms * 1e3, 1),
                              "roofline_us": round(roof * 1e3, 1), "frac": round(roof / ms, 3),
                              "like": like}), flush=True)


if __name__ == "__main__":
    main()
