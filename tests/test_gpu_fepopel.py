"""Fepopel on the GPU: its kernels against the torch formulation, the engine's step against the
oracle in both dtypes (caches per layer run, portions, mixed batches, CUDA graphs), generation, and
the trace runner as a command."""
import json
import os
import subprocess

import pytest
import torch

import fepopel_oracle as O
from fepopel_cases import (CONFIGS, build, chunked, clear_choices, dense, errors, greedy,
                           latent, mixed_steps, model_config, moe, oracle, paged_batch,
                           peaked_model, portions, replayer, run, spread, tokens_for)

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF16 = torch.float32, torch.bfloat16


def _close(got, want, dtype, scale=None):
    got, want = got.float().cpu(), want.float()
    assert torch.isfinite(got).all()
    lim = (0.02 if dtype == BF16 else 2e-5) * (scale or max(1.0, want.abs().max().item()))
    assert (got - want).abs().max().item() < lim, ((got - want).abs().max().item(), lim)


def _status():
    from vllm_gcu_b200.ops import _native
    torch.cuda.synchronize()
    _native.check_status()


def _cuda(x):
    if isinstance(x, dict):
        return {k: _cuda(v) for k, v in x.items()}
    return x.cuda() if torch.is_tensor(x) else x


# -- residual stream --------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,H", [(3, 72), (2, 37), (300, 2048), (5, 7168), (1, 13000)])
def test_residual_kernels(T, H, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    g = torch.Generator().manual_seed(H)
    e = torch.randn(T, H, generator=g).to(dtype)
    x, step, w, wb = (torch.randn(*s, generator=g) for s in ((T, H), (H,), (H,), (H,)))
    for kw in (dict(), dict(step=step), dict(weight=w, eps=1e-3), dict(step=step, weight=w, eps=1e-3)):
        got, want = C.start_rows(e.cuda(), 1.7, **_cuda(kw)), ref.start_rows(e.float(), 1.7, **kw)
        _close(got[0], want[0], F32)
        _close(got[1], want[1], dtype)
    k, Hp = 3, -(-H // 64) * 64
    rows = torch.randn(T * k + 5, Hp, generator=g).to(dtype)
    pos = torch.randperm(T * k + 5, generator=g)[:T * k].int()
    pos[0] = -1
    row_w, gate = torch.rand(T, k, generator=g), torch.randn(T, 16, generator=g)
    shared = torch.randn(T, H, generator=g).to(dtype)
    dense_y = torch.randn(T, H, generator=g).to(dtype)
    routed = dict(pos_of=pos, row_w=row_w)
    for y, kw in ((dense_y, dict(step=step)), (rows, routed), (rows, {**routed, "shared": shared}),
                  (rows, {**routed, "shared": shared, "gate": gate[:, 8], "step": step})):
        for final in (None, w):
            out, lo = torch.empty(T, H), torch.empty(T, H)
            kr = {n: v.float() if torch.is_tensor(v) and v.dtype == BF16 else v
                  for n, v in kw.items()}
            ref.add_normed(x, y.float(), wb, None, 1e-4, lo, out=out, layer_norm=False,
                           final_weight=final, **kr)
            kg = _cuda(kw)
            if "gate" in kg:
                kg["gate"] = gate.cuda()[:, 8]
            gx, glo = x.cuda(), torch.empty(T, H, dtype=dtype, device="cuda")
            C.add_normed(gx, y.cuda(), wb.cuda(), None, 1e-4, glo, out=gx, layer_norm=False,
                         final_weight=_cuda(final), **kg)
            _close(gx, out, F32)
            _close(glo, lo, dtype)
    u = torch.randn(T, H, generator=g).to(dtype)
    _close(C.ungated_act(u.cuda(), "relu2"), u.float().clamp(min=0).square(), dtype)


# -- squared-ReLU products --------------------------------------------------------------
@pytest.mark.parametrize("M,N,K", [(1, 1408, 2048), (64, 2816, 2048), (7, 40, 72), (200, 512, 256),
                                   (129, 96, 64), (1024, 1536, 512), (4096, 4096, 1024),
                                   (64, 13, 24)])
def test_gemm_with_squared_relu(M, N, K):
    from vllm_gcu_b200.ops import cuda as C
    g = torch.Generator().manual_seed(N)
    a, b = torch.randn(M, K, generator=g).to(BF16), (torch.randn(N, K, generator=g) * K ** -0.5).to(BF16)
    got = C.gemm_bf16(a.cuda(), b.cuda(), epilogue=C.EPI_RELU2)
    _status()
    want = (a.cuda().float() @ b.cuda().float().t()).clamp(min=0).square().cpu()
    _close(got, want, BF16)


@pytest.mark.parametrize("M,N,K", [(64, 72, 7168), (1, 40, 2048), (128, 264, 4096), (100, 8, 8192),
                                   (3, 24, 256), (129, 72, 4096), (5, 1024, 5120)])
def test_gemm_with_fp32_results(M, N, K):
    from vllm_gcu_b200.ops import cuda as C
    g = torch.Generator().manual_seed(N)
    a, b = torch.randn(M, K, generator=g).to(BF16), (torch.randn(N, K, generator=g) * K ** -0.5).to(BF16)
    got = C.gemm_bf16(a.cuda(), b.cuda(), epilogue=C.EPI_FP32)
    _status()
    assert got.dtype == F32
    _close(got, (a.cuda().double() @ b.cuda().double().t()).float().cpu(), F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,F,E,k,S,T", [(72, 24, 5, 2, 20, 1), (100, 36, 4, 1, 0, 70),
                                         (256, 128, 16, 6, 96, 300), (37, 11, 3, 3, 5, 9),
                                         (512, 320, 9, 2, 64, 129)])
def test_experts_and_shared_expert(H, F, E, k, S, T, dtype):
    from vllm_gcu_b200.layers.moe import GatedSharedMoE
    from vllm_gcu_b200.ops import cuda as C
    g = torch.Generator().manual_seed(H)
    m = GatedSharedMoE(E, k, 1.6, H, F, S, dtype, "cuda", "x")
    shapes = {"router": (E, H), **{f"e{e}.up": (F, H) for e in range(E)},
              **{f"e{e}.down": (H, F) for e in range(E)}}
    if S:
        shapes.update({"shared.up": (S, H), "shared.down": (H, S), "shared.sg": (1, H)})
    w = {n: (torch.randn(*s, generator=g) * s[1] ** -0.5).to(BF16) for n, s in shapes.items()}
    w["router"] = (torch.randn(E, H, generator=g) * 4 * H ** -0.5).to(BF16)
    assert all(m.load(n, t) for n, t in w.items())
    for mod in m.modules():
        if mod is not m and hasattr(mod, "finalize"):
            mod.finalize()
    h = torch.randn(T, H, generator=g).to(dtype)
    y, rows = m(h.cuda())
    x, lo = torch.zeros(T, H, device="cuda"), torch.empty(T, H, dtype=dtype, device="cuda")
    one = torch.ones(H, device="cuda")
    C.add_normed(x, y, one, None, 1e-6, lo, layer_norm=False, **rows)
    _status()
    want = O.moe(h.double(), {n: t.double() for n, t in w.items()}, k, 1.6)
    e = (lo.float().cpu() - O.rms(want, torch.ones(H), 1e-6).float()).pow(2).mean(-1).sqrt()
    # a row may choose another expert where rounding decides a close call
    assert (e < (0.03 if dtype == BF16 else 2e-5)).float().mean() >= (0.97 if dtype == BF16 else 1.0)


# -- attention --------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("Hq,Hkv,D,VD,DC", [(4, 2, 20, 28, 28), (3, 1, 7, 5, 9), (16, 4, 128, 128, 128),
                                            (6, 3, 64, 48, 64), (2, 2, 200, 512, 512),
                                            (1, 1, 512, 16, 512)])
def test_head_norm_cache(Hq, Hkv, D, VD, DC, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    g = torch.Generator().manual_seed(D)
    T, nb, bs = 13, 4, 8
    wide = (torch.randn(T, Hq * D + Hkv * (D + VD) + 24, generator=g) * 2).to(dtype)
    at = [8, 8 + Hq * D, 8 + (Hq + Hkv) * D]
    cut = lambda t: (t[:, at[0]:at[1]], t[:, at[1]:at[2]], t[:, at[2]:at[2] + Hkv * VD])  # noqa: E731
    qw, kw = torch.randn(D, generator=g), torch.randn(D, generator=g)
    slots = torch.randperm(nb * bs, generator=g)[:T].long()
    slots[3] = -1
    kc, vc = (torch.full((nb, bs, Hkv, DC), 3.0).to(dtype) for _ in range(2))
    gk, gv = kc.cuda(), vc.cuda()
    got = C.head_norm_cache(*cut(wide.cuda()), qw.cuda(), kw.cuda(), 1e-3, slots.cuda(), gk, gv, D)
    _status()
    fk, fv = kc.float(), vc.float()
    want = ref.head_norm_cache(*cut(wide.float()), qw, kw, 1e-3, slots, fk, fv, D)
    for a, b in ((got, want), (gk, fk), (gv, fv)):
        _close(a, b, dtype)


SHAPES = [(49, 1), (130, 1), (0, 1), (300, 1), (131, 70), (41, 2), (300, 300), (513, 200)]


def _shaped(Hq, Hkv, D, chunk, dtype, seed, bs=16):
    ql, sl = [n for _, n in SHAPES], [n for n, _ in SHAPES]
    return paged_batch(Hq, Hkv, D, ql, sl, chunk, dtype, bs, seed), 4


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("chunk,softcap", [(0, 0.0), (24, 5.0), (64, 0.0), (100, 30.0), (1, 3.0),
                                           (0, 8.0)])
@pytest.mark.parametrize("Hq,Hkv,D,OD", [(3, 1, 20, 12), (4, 2, 160, 160)])
def test_general_attention_with_chunks_and_caps(Hq, Hkv, D, OD, chunk, softcap, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    (q, kc, vc, bt, s, cu), nd = _shaped(Hq, Hkv, D, chunk, dtype, D + chunk, bs=8)
    sink = torch.linspace(-2.0, 9.0, Hq)
    kw = dict(softcap=softcap, chunk=chunk, out_dim=OD)
    rest = cu[nd:] - cu[nd]
    for sk in (None, sink):
        buf = torch.full((q.shape[0], Hq * OD + 8), 2.0, dtype=dtype, device="cuda")
        C.any_attention(q.cuda(), kc.cuda(), vc.cuda(), bt.cuda(), s.cuda(), nd, rest.cuda(),
                        D ** -0.5, _cuda(sk), out=buf[:, :Hq * OD].unflatten(1, (Hq, OD)), **kw)
        _status()
        want = ref.any_attention(q.float(), kc.float(), vc.float(), bt, s, nd, rest, D ** -0.5, sk,
                                 **kw)
        _close(buf[:, :Hq * OD].unflatten(1, (Hq, OD)), want, dtype)
        assert (buf[:, Hq * OD:] == 2.0).all()


@pytest.mark.parametrize("chunk,softcap", [(24, 5.0), (64, 30.0), (100, 0.0), (1, 3.0), (0, 8.0),
                                           (150, 50.0), (128, 20.0), (1000, 12.0), (0, 0.0)])
@pytest.mark.parametrize("Hq,Hkv,D,OD", [(4, 2, 64, 48), (16, 1, 96, 72), (8, 2, 128, 128),
                                         (6, 6, 128, 100), (2, 1, 64, 13)])
def test_tensor_core_attention_with_chunks_and_caps(Hq, Hkv, D, OD, chunk, softcap):
    """Single tokens (with and without context splits) and portions, at the edges of chunks, pages
    and tiles."""
    from vllm_gcu_b200.ops import cuda as C, ref
    (q, kc, vc, bt, s, cu), nd = _shaped(Hq, Hkv, D, chunk, BF16, D + chunk)
    sink = torch.linspace(-2.0, 9.0, Hq)
    kw = dict(softcap=softcap, chunk=chunk, out_dim=OD)
    rest = cu[nd:] - cu[nd]
    gq, gk, gv, gb, gs = (t.cuda() for t in (q, kc, vc, bt, s))
    for sk in (None, sink):
        want = ref.any_attention(q.float(), kc.float(), vc.float(), bt, s, nd, rest, D ** -0.5, sk,
                                 **kw)
        pitch = Hq * OD + (8 if (Hq * OD) % 8 == 0 else 3)
        buf = torch.full((q.shape[0], pitch), 2.0, dtype=BF16, device="cuda")
        out = buf[:, :Hq * OD].unflatten(1, (Hq, OD))
        for splits in (1, 3):
            out[:nd].fill_(5.0)
            C.paged_decode(gq[:nd], gk, gv, gb[:nd], gs[:nd], D ** -0.5, out=out[:nd],
                           num_splits=splits, sink=_cuda(sk), **kw)
            _status()
            _close(out[:nd], want[:nd], BF16)
        tiles = sum(-(-n // 128) for _, n in SHAPES[nd:])
        done = C.fmha_prefill_sink(gq[nd:], gk, gv, gb[nd:], rest.cuda(), gs[nd:], D ** -0.5, tiles,
                                   _cuda(sk), out=out[nd:], **kw)
        _status()
        assert done is not None
        _close(out[nd:], want[nd:], BF16)
        assert (buf[:, Hq * OD:] == 2.0).all()


def _latent_batch(N, L, R, W, q_lens, seq_lens, dtype, bs=16, seed=0):
    """Latent queries that each match one cached row, near or far; the first row a query may not see
    matches best."""
    g = torch.Generator().manual_seed(seed)
    B = len(q_lens)
    mb = max(1, -(-max(seq_lens) // bs)) + 1
    nb = B * mb + 3
    cache = torch.randn(nb, bs, W, generator=g)
    cache[..., L + R:] = 0
    bt = (torch.randperm(nb - 1, generator=g)[:B * mb] + 1).view(B, mb).int()
    rows = []
    for b, (ql, n) in enumerate(zip(q_lens, seq_lens)):
        for i in range(ql):
            seen = n - ql + i + 1
            for a in range(N):
                cand = [c for c in (0, seen - 1, seen // 2, 15, 16, 63, 64, 127, 128) if 0 <= c < seen]
                row = torch.randn(W, generator=g) * 0.3
                if cand:
                    p = cand[(a + i) % len(cand)]
                    k = cache[bt[b, p // bs], p % bs]
                    row = k * (6.0 * W ** 0.5 / (k @ k))
                    if seen < n:
                        f = cache[bt[b, seen // bs], seen % bs]
                        row = row + f * (9.0 * W ** 0.5 / (f @ f))
                rows.append(row)
    q = torch.stack(rows).view(sum(q_lens), N, W)
    cu = torch.tensor([0] + list(torch.tensor(q_lens).cumsum(0)), dtype=torch.int32)
    return (q.to(dtype), cache.to(dtype), bt, torch.tensor(seq_lens, dtype=torch.int32), cu)


@pytest.mark.parametrize("N,L,R", [(1, 30, 2), (3, 96, 20), (6, 90, 64), (12, 240, 16), (33, 320, 64),
                                   (128, 512, 64), (16, 500, 12), (40, 64, 64), (20, 384, 0)])
def test_tensor_core_latent_attention_with_sinks_and_gates(N, L, R):
    from vllm_gcu_b200.ops import cuda as C, ref
    W, V = -(-(L + R) // 64) * 64, -(-L // 64) * 64
    scale = 2.0 * W ** -0.5
    sink = torch.linspace(-3.0, 12.0, N)
    for decode, ql, sl, splits in (
            (True, [1] * 6, [1, 17, 64, 65, 300, 0], 1), (True, [1] * 4, [130, 16, 700, 77], 4),
            (False, [40, 7, 130, 1], [40, 100, 130, 9], 1), (False, [33, 2], [333, 500], 3)):
        q, cache, bt, s, cu = _latent_batch(N, L, R, W, ql, sl, BF16, seed=N)
        wide = torch.randn(sum(ql), N + 11, generator=torch.Generator().manual_seed(1)).to(BF16)
        for sk, use_gate in ((sink, True), (None, True), (sink, False)):
            got = C.mla_attention(q.cuda(), cache.cuda(), bt.cuda(), s.cuda(),
                                  None if decode else cu.cuda(), sum(-(-x // (128 // N)) for x in ql),
                                  max(sl), scale, splits=splits, L=V, sink=_cuda(sk),
                                  gate=wide.cuda()[:, 3:3 + N] if use_gate else None)
            _status()
            want = ref.latent_attention(q.float(), cache.float(), bt, ql, sl, scale, V, sk,
                                        wide[:, 3:3 + N] if use_gate else None)
            _close(got, want, BF16)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("N,L,R", [(1, 3, 2), (3, 30, 8), (9, 90, 12), (17, 500, 64), (2, 1000, 6)])
def test_general_latent_attention_with_sinks_and_gates(N, L, R, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    W = -(-(L + R) // 4) * 4
    scale = 2.0 * W ** -0.5
    ql, sl, nd = [1, 1, 1, 40, 2, 65], [1, 300, 0, 40, 99, 200], 3
    q, cache, bt, s, cu = _latent_batch(N, L, R, W, ql, sl, dtype, bs=8, seed=W)
    sink = torch.linspace(-3.0, 12.0, N)
    wide = torch.randn(sum(ql), N + 5, generator=torch.Generator().manual_seed(1)).to(dtype)
    got = C.latent_attention(q.cuda(), cache.cuda(), bt.cuda(), s.cuda(), nd, (cu[nd:] - cu[nd]).cuda(),
                             scale, sink=sink.cuda(), gate=wide.cuda()[:, 2:2 + N])
    _status()
    _close(got, ref.latent_attention(q.float(), cache.float(), bt, ql, sl, scale, W, sink,
                                     wide[:, 2:2 + N]), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("N,dim,L,R", [(3, 12, 36, 6), (2, 5, 9, 2), (16, 128, 512, 64), (1, 8, 30, 34),
                                       (5, 7, 1100, 12)])
def test_latent_cache_with_rotated_part(N, dim, L, R, dtype):
    from vllm_gcu_b200.layers.basic import build_cos_sin_cache
    from vllm_gcu_b200.ops import cuda as C, ref
    g = torch.Generator().manual_seed(L)
    T, bs, nb = 19, 16, 6
    W = -(-(L + R) // 64) * 64
    nq = N * (dim + R)
    wide = torch.randn(T, nq + L + R + 16, generator=g).to(dtype)
    cut = lambda t: (t[:, 8:8 + nq], t[:, 8 + nq:8 + nq + L + R])  # noqa: E731
    nw = torch.randn(L, generator=g).to(dtype)
    cs = build_cos_sin_cache(R, 4000, 300.0, dtype=torch.float64).float()
    pos = torch.randint(0, 4000, (T,), generator=g)
    slots = torch.randperm(nb * bs, generator=g)[:T].long()
    slots[5] = -1
    cache, q_lat = torch.full((nb, bs, W), 3.0).to(dtype), torch.randn(T, N, W, generator=g).to(dtype)
    gc, gq = cache.cuda(), q_lat.cuda()
    q, kv = cut(wide.cuda())
    C.latent_cache(kv, nw.cuda(), 1e-3, gc, slots.cuda(), cos_sin=cs.cuda(), positions=pos.cuda(), q=q,
                   q_lat=gq)
    _status()
    fc, fq = cache.float(), q_lat.float()
    q, kv = cut(wide.float())
    ref.latent_cache(kv, nw.float(), 1e-3, fc, slots, cos_sin=cs, positions=pos, q=q, q_lat=fq)
    _close(gc, fc, dtype)
    _close(gq, fq, dtype)
    keep = [c for c in range(W) if not L <= c < L + R]
    assert torch.equal(gq.cpu()[..., keep], q_lat[..., keep])


# -- the engine's step ------------------------------------------------------------------
GPU_CONFIGS = {**CONFIGS,
               # more heads than a tile has rows, groups larger than the decode kernel's, heads and
               # latent rows wider than the tensor-core kernels'
               "big": model_config(120, 128, [
                   latent(130, 8, 4, 8, 60, 1e3, 0.3, moe(4, 2, 64, 32, 1.3)),
                   chunked(34, 2, 40, 24, 70, 0.2, 10.0, dense(64)),
                   latent(4, 32, 16, 48, 600, 1e4, 0.18, moe(3, 1, 48)),
                   chunked(4, 2, 136, 72, 33, 0.1, 15.0)], (1, 3, 2))}


def _check(got, want, dtype, clear=None, what=""):
    e = errors(got, want)
    if dtype == "float32":
        assert e.max() < 2e-4, (what, e.max())
    else:
        # rounding; it may decide a close call between experts, and later rows see such a row
        assert e[clear].numel() == 0 or e[clear].max() < 0.15, (what, e)
        assert (e[clear] > 0.06).float().mean() <= 0.03 or int((e[clear] > 0.06).sum()) <= 1, (what, e)
        assert (e > 0.06).float().mean() <= 0.15 or int((e > 0.06).sum()) <= 1, (what, e)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(GPU_CONFIGS))
def test_portions_and_decoding(tmp_path, name, dtype):
    cfg, w, path = build(tmp_path, name, configs=GPU_CONFIGS)
    toks = tokens_for(cfg, 150)
    want, clear = oracle(cfg, w, {"a": toks})["a"], clear_choices(cfg, w, toks)
    assert clear.float().mean() > 0.25
    rp = replayer(path, "cuda", dtype, max_tokens=192)
    for sizes in ([150], [2, 3, 64, 1], [31, 2, 1], [100] + [1] * 50):
        got = run(rp, {"a": toks}, [[("a", n)] for n in portions(150, sizes)])["a"]
        _check(got, want, dtype, clear, sizes)
    assert rp.engine.runner.graph_launches > 0           # decoded through CUDA graphs
    _status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["uneven", "wide"])
def test_mixed_batches_and_reused_blocks(tmp_path, name, dtype):
    cfg, w, path = build(tmp_path, name, seed=5)
    prompts = {f"r{i}": tokens_for(cfg, n, i) for i, n in
               enumerate((1, 40, 2, 65, 17, 130, 33, 3, 64, 16))}
    want = oracle(cfg, w, prompts)
    rp = replayer(path, "cuda", dtype, max_tokens=384)
    got = run(rp, prompts, mixed_steps(prompts))
    for k in prompts:
        _check(got[k], want[k], dtype, clear_choices(cfg, w, prompts[k]), k)
    assert rp.engine.scheduler.kv.pool.num_free_blocks == rp.engine.scheduler.kv.pool.num_blocks


def test_far_keys_and_chunk_edges(tmp_path):
    cfg, w, path = build(tmp_path, "uneven", seed=4, weights=peaked_model)
    n = 268                                 # the last chunk of 24 starts at 264
    rp = replayer(path, "cuda", "float32", max_tokens=320)
    for p in (0, 1, 15, 16, 63, 64, 127, 255, 263, 264, 265):
        toks = tokens_for(cfg, n, 7)
        toks[p] = (toks[p] + 1) % cfg["vocab"]
        want = O.forward(cfg, w, toks)
        for sizes in ([n], [n - 6] + [1] * 6):
            got = run(rp, {"a": toks}, [[("a", c)] for c in portions(n, sizes)])["a"]
            assert errors(got, want).max() < 2e-3, (p, sizes)


def test_long_decoding(tmp_path):
    cfg, w, path = build(tmp_path, "ones", seed=7)
    prompts = {"a": tokens_for(cfg, 300, 1), "b": tokens_for(cfg, 260, 2)}
    want = oracle(cfg, w, prompts)
    steps = spread([("a", 2)] + [("a", 1)] * 298, [("b", 1)] * 260)
    got = run(replayer(path, "cuda", "float32", max_tokens=640), prompts, steps)
    for k in prompts:
        _check(got[k], want[k], "float32", what=k)


# -- generation and command -------------------------------------------------------------
def test_greedy_generation(tmp_path):
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    cfg, w, path = build(tmp_path, "uneven", seed=9)
    prompts = [tokens_for(cfg, n, 20 + n) for n in (1, 18, 37, 50)]
    prompts.append(prompts[-1][:48] + prompts[0])        # shares full blocks with another
    want = [greedy(cfg, w, p, 12) for p in prompts]
    sp = SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True)
    for kw in (dict(async_scheduling=True), dict(max_num_batched_tokens=16),
               dict(enforce_eager=True), dict(num_gpu_blocks=7, num_cpu_blocks=16),
               dict(speculative_method="ngram", num_speculative_tokens=2)):
        llm = LLM(path, dtype="float32", **{**dict(max_num_seqs=4, max_model_len=128,
                                                   num_gpu_blocks=64), **kw})
        assert [o.outputs[0].token_ids for o in llm.generate(prompts, sp)] == want, kw
        assert [o.outputs[0].token_ids for o in llm.generate(prompts, sp)] == want, kw
    llm = LLM(path, dtype="bfloat16", max_num_seqs=4, max_model_len=128)    # profiled cache size
    outs = llm.generate(prompts, sp)
    assert all(len(o.outputs[0].token_ids) == 12 for o in outs)


def test_trace_run_command(tmp_path):
    cfg, w, path = build(tmp_path, "wide", seed=3)
    toks = tokens_for(cfg, 40)
    want = O.forward(cfg, w, toks)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[30:39], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[39:], "want": [0]}], "end": ["x"]}]
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype",
                        "float32", "--out", str(out), "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    done = [x for x in p.stdout.splitlines() if x.startswith("done")]
    assert done == ["done 0", "done 1", "done 2"]
    import numpy as np
    got = np.concatenate([np.fromfile(out / f, dtype="<f4").reshape(-1, cfg["vocab"])
                          for f in ("0.f32", "2.f32")])
    assert errors(torch.from_numpy(got), want[[0, 29, 39]]).max() < 2e-4
