"""Sapapel on the GPU: its kernels against the torch formulation, the engine's step against the
oracle in both dtypes (cache, block state, portions, mixed batches, CUDA graphs), generation, and
the trace runner as a command."""
import json
import os
import subprocess
import sys

import pytest
import torch

import sapapel_oracle as O
from sapapel_cases import (CONFIGS, errors, layer, mixed_steps, model_config, oracle,
                           peaked_weights, portions, replayer, run, tokens_for, write_checkpoint)

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# -- kernels ----------------------------------------------------------------------------
def _batch(W, N, q_lens, seq_lens, dtype, bs=16, seed=0, peaked=True):
    """Paged latent rows and queries.  With ``peaked`` every query row is a multiple of one key
    row, far or near, first, last or at the edge of a page or a tile, so that one score stands
    out; the last key that a row may not see is made the best match of all."""
    g = torch.Generator().manual_seed(seed)
    B = len(q_lens)
    mb = max(1, -(-max(seq_lens) // bs)) + 1
    nb = B * mb + 3
    cache = torch.randn(nb, bs, W, generator=g)
    bt = (torch.randperm(nb - 1, generator=g)[:B * mb] + 1).view(B, mb).int()
    rows = []
    for b, (ql, n) in enumerate(zip(q_lens, seq_lens)):
        for i in range(ql):
            seen = n - ql + i + 1
            for a in range(N):
                if not peaked or seen <= 0:
                    rows.append(torch.randn(W, generator=g) * 0.5)
                    continue
                cand = [0, seen - 1, seen // 2, 15, 16, 17, 31, 63, 64, 65, 127, 128]
                cand = [c for c in cand if c < seen]
                p = cand[(a + i) % len(cand)]
                k = cache[bt[b, p // bs], p % bs]
                row = k * (6.0 * W ** 0.5 / (k @ k))
                if seen < n:                     # a key of the future matches better
                    f = cache[bt[b, seen // bs], seen % bs]
                    row = row + f * (9.0 * W ** 0.5 / (f @ f))
                rows.append(row)
    q = torch.stack(rows).view(sum(q_lens), N, W)
    cu = torch.tensor([0] + list(torch.tensor(q_lens).cumsum(0)), dtype=torch.int32)
    return (q.to(dtype), cache.to(dtype), bt, torch.tensor(seq_lens, dtype=torch.int32), cu)


def _close(got, want, dtype):
    err = (got.float().cpu() - want).abs().max().item()
    lim = (0.02 if dtype == torch.bfloat16 else 1e-5) * max(1.0, want.abs().max().item())
    assert err < lim, (err, lim)


@pytest.mark.parametrize("N,L,W", [(1, 64, 64), (3, 128, 128), (5, 192, 192), (12, 256, 256),
                                   (20, 320, 320), (33, 384, 384), (48, 448, 448), (100, 512, 512),
                                   (128, 512, 512), (16, 512, 576), (7, 64, 128), (128, 256, 320)])
def test_tensor_core_latent_attention_shapes(N, L, W):
    from vllm_gcu_b200.ops import _native, cuda as C, ref
    scale = 2.0 * W ** -0.5
    dev = "cuda"
    for decode, ql, sl, splits in (
            (True, [1] * 6, [1, 17, 64, 65, 300, 0], 1), (True, [1] * 4, [130, 16, 700, 77], 4),
            (False, [40, 7, 130, 1], [40, 100, 130, 9], 1), (False, [33, 2], [333, 500], 3)):
        q, cache, bt, s, cu = _batch(W, N, ql, sl, torch.bfloat16, seed=N)
        tq = 128 // N
        got = C.mla_attention(q.to(dev), cache.to(dev), bt.to(dev), s.to(dev),
                              None if decode else cu.to(dev), sum(-(-x // tq) for x in ql),
                              max(sl), scale, splits=splits, L=L)
        torch.cuda.synchronize()
        _native.check_status()
        _close(got, ref.latent_attention(q.float(), cache.float(), bt, ql, sl, scale, L),
               torch.bfloat16)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("N,W", [(1, 4), (3, 36), (9, 100), (8, 256), (17, 516), (2, 1024)])
def test_general_latent_attention(N, W, dtype):
    from vllm_gcu_b200.ops import _native, cuda as C, ref
    scale, dev = 2.0 * W ** -0.5, "cuda"
    ql, sl, nd = [1, 1, 1, 40, 2, 65], [1, 300, 0, 40, 99, 200], 3
    q, cache, bt, s, cu = _batch(W, N, ql, sl, dtype, bs=8, seed=W)
    got = C.latent_attention(q.to(dev), cache.to(dev), bt.to(dev), s.to(dev), nd,
                             (cu[nd:] - cu[nd]).to(dev), scale)
    torch.cuda.synchronize()
    _native.check_status()
    _close(got, ref.latent_attention(q.float(), cache.float(), bt, ql, sl, scale, W), dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,L", [(72, 36), (101, 30), (2048, 512)])
def test_shift_and_cache_kernels(H, L, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    g = torch.Generator().manual_seed(H)
    bs, nb = 16, 24
    nd, lens, starts = 3, [1, 1, 1, 2, 33, 16], [0, 16, 37, 15, 7, 32]
    T, pad = sum(lens), 2                        # rows behind the last request: no slot
    mu, x = torch.rand(H, generator=g), torch.randn(T + pad, H, generator=g)
    state = torch.randn(nb, H, generator=g)
    bt = torch.randperm(nb, generator=g)[:6 * 4].view(6, 4).int()
    pos = torch.cat([torch.arange(a, a + n) for a, n in zip(starts, lens)] + [torch.zeros(pad)]).long()
    slots = torch.cat([bt[r][torch.arange(a, a + n) // bs].long() * bs + torch.arange(a, a + n) % bs
                       for r, (a, n) in enumerate(zip(starts, lens))] + [torch.full((pad,), -1)]).long()
    cu = torch.tensor([0] + lens[nd:]).cumsum(0).int()
    wide = torch.randn(T + pad, L + 9, generator=g).to(dtype)       # the latent is a slice
    nw = torch.randn(L, generator=g).to(dtype)
    W = -(-L // 64) * 64
    cache = torch.full((nb, bs, W), 3.0).to(dtype)
    d = lambda t: t.cuda()  # noqa: E731
    want = ref.token_shift(x, mu, torch.float32, state, bt, pos, nd, cu, bs)
    dstate, dcache = d(state), d(cache)
    got = C.token_shift(d(x), d(mu), dtype, dstate, d(bt), d(pos), nd, d(cu), bs)
    _close(got[:T], want[:T], dtype)
    C.latent_cache(d(wide)[:, 5:5 + L], d(nw), 1e-3, dcache, d(slots), d(x), dstate, nd, d(cu))
    ref_cache = cache.float()
    ref.latent_cache(wide[:, 5:5 + L].float(), nw.float(), 1e-3, ref_cache, slots, x, state, nd, cu)
    _close(dcache, ref_cache, dtype)
    assert torch.equal(dstate.cpu(), state)
    assert torch.allclose(C.token_shift(d(x[:1]), d(mu), torch.float32).cpu(),
                          x[:1] * (1 - mu), atol=1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H,n", [(1, 72, 1), (3, 101, 6), (300, 256, 4), (2, 7168, 9)])
def test_post_norm_kernel(T, H, n, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    g = torch.Generator().manual_seed(H)
    k = 3
    x, hist = torch.randn(T, H, generator=g), torch.randn(n + 1, T, H, generator=g)
    gain, fgain, w = torch.tensor(1.3), torch.tensor(0.6), torch.randn(n + 1, generator=g)
    Hp = -(-H // 64) * 64
    rows = torch.randn(T * k + 5, Hp, generator=g).to(dtype)
    pos = torch.randperm(T * k + 5, generator=g)[:T * k].int()
    pos[-1] = -1
    dense = torch.randn(T, H, generator=g).to(dtype)
    d = lambda t: None if t is None else t.cuda()  # noqa: E731
    for y, p, kk in ((dense, None, 0), (rows, pos, k)):
        for use_hist, final in ((False, None), (True, None), (True, fgain)):
            def call(mod, dev):
                f = (lambda t: t) if mod is ref else d
                o = {s: torch.full((T, H), 5.0, dtype=torch.float32 if s != "lo" or mod is ref
                                   else dtype, device=dev) for s in ("res", "avg", "lo")}
                mod.post_norm(f(x), f(y.float() if mod is ref else y), f(gain), 1.9, 1e-4,
                              pos_of=f(p) if p is not None else None, k=kk, res=o["res"],
                              hist=f(hist) if use_hist else None, n=n, weights=f(w),
                              avg=o["avg"] if use_hist else None,
                              final_gain=f(final) if final is not None else None, lo=o["lo"])
                return o
            a, b = call(C, "cuda"), call(ref, "cpu")
            for s in ("res", "avg"):
                _close(a[s], b[s], torch.float32)
            _close(a["lo"], b["lo"], dtype)
    # the average may overwrite its input
    xi = d(x)
    C.post_norm(xi, d(dense), d(gain), 1.9, 1e-4, hist=d(hist), n=n, weights=d(w), avg=xi)
    want = torch.empty(T, H)
    ref.post_norm(x, dense.float(), gain, 1.9, 1e-4, hist=hist, n=n, weights=w, avg=want)
    _close(xi, want, torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,F,E,k,T", [(72, 24, 5, 2, 1), (100, 36, 4, 1, 70), (256, 128, 16, 6, 300),
                                       (37, 11, 3, 3, 9), (512, 320, 9, 2, 129)])
def test_input_weighted_experts(H, F, E, k, T, dtype):
    from vllm_gcu_b200.layers.moe import InputWeightedMoE
    from vllm_gcu_b200.ops import _native, cuda as C, ref
    g = torch.Generator().manual_seed(H)
    moe = InputWeightedMoE(E, H, F, dtype, "cuda")
    w = {}
    for e in range(E):
        for n, s in (("gate", (F, H)), ("up", (F, H)), ("down", (H, F))):
            w[f"e{e}.{n}"] = (torch.randn(*s, generator=g) * s[1] ** -0.5).to(dtype)
            moe.load_expert_weight(e, n, w[f"e{e}.{n}"])
    moe.finalize()
    x = torch.randn(T, H, generator=g) * 3
    z = torch.randn(T, E, generator=g)
    s, ids = C.moe_topk(z.cuda(), k, False, sigmoid=True)
    y, pos = moe(x.cuda(), s, ids)
    got = torch.empty(T, H, dtype=torch.float32, device="cuda")
    one = torch.ones((), device="cuda")
    C.post_norm(torch.zeros(T, H, device="cuda"), y, one, 1.0, 1e-6, pos_of=pos, k=k, res=got)
    torch.cuda.synchronize()
    _native.check_status()
    ws, wi = torch.sigmoid(z).topk(k, -1)
    want = torch.zeros(T, H)
    for t in range(T):
        for j in range(k):
            e = int(wi[t, j])
            want[t] += O.expert((ws[t, j] * x[t])[None], *(w[f"e{e}.{n}"].float()
                                                         for n in ("gate", "up", "down")))[0]
    _close(got, ref.scalar_rms_norm(want, torch.ones(()), 1e-6), dtype)


# -- the engine's step ------------------------------------------------------------------
GPU_CONFIGS = {**CONFIGS,
               # latent rows wider than the tensor-core kernel's and more heads than a tile's rows
               "big": model_config(120, 128, 1.4, 1e-5, [layer(130, 8, 8, 96, 0.3, 4, 2, 64),
                                                         layer(4, 32, 48, 600, 0.18, 3, 1, 48),
                                                         layer(40, 16, 24, 512, 0.25)])}


def _build(tmp_path, name, seed=0, sharp=None):
    cfg = GPU_CONFIGS[name]
    w = O.random_model(cfg, seed) if sharp is None else peaked_weights(cfg, seed, sharp)
    return cfg, w, write_checkpoint(tmp_path / name, cfg, w)


def _check(got, want, dtype, what=""):
    e = errors(got, want)
    if dtype == "float32":
        assert e.max() < 2e-4, (what, e.max())
    else:
        # rounding, and at most a few rows where it decides a close call between experts
        assert (e > 0.06).float().mean() <= 0.03 or int((e > 0.06).sum()) <= 1, (what, e)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(GPU_CONFIGS))
def test_portions_and_decoding(tmp_path, name, dtype):
    cfg, w, path = _build(tmp_path, name)
    toks = tokens_for(cfg, 150)
    want = oracle(cfg, w, {"a": toks})["a"]
    rp = replayer(path, "cuda", dtype, max_tokens=192)
    for sizes in ([150], [2, 3, 64, 1], [31, 2, 1], [100] + [1] * 50):
        got = run(rp, {"a": toks}, [[("a", n)] for n in portions(150, sizes)])["a"]
        _check(got, want, dtype, sizes)
    assert rp.engine.runner.graph_launches > 0           # decoded through CUDA graphs
    from vllm_gcu_b200.ops import _native
    _native.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["uneven", "wide"])
def test_mixed_batches_and_reused_blocks(tmp_path, name, dtype):
    cfg, w, path = _build(tmp_path, name, seed=5)
    prompts = {f"r{i}": tokens_for(cfg, n, i) for i, n in
               enumerate((1, 40, 2, 65, 17, 130, 33, 3, 64, 16))}
    want = oracle(cfg, w, prompts)
    rp = replayer(path, "cuda", dtype, max_tokens=384)
    got = run(rp, prompts, mixed_steps(prompts))
    for k in prompts:
        _check(got[k], want[k], dtype, k)
    assert rp.engine.scheduler.kv.pool.num_free_blocks == rp.engine.scheduler.kv.pool.num_blocks


def test_far_keys(tmp_path):
    cfg, w, path = _build(tmp_path, "uneven", seed=4, sharp=6.0)
    n = 300
    rp = replayer(path, "cuda", "float32", max_tokens=320)
    for p in (0, 1, 15, 16, 31, 63, 64, 127, 255):
        toks = tokens_for(cfg, n, 7)
        toks[p] = (toks[p] + 1) % cfg["vocab"]
        want = O.forward(cfg, w, toks)
        for sizes in ([n], [n - 6] + [1] * 6):
            got = run(rp, {"a": toks}, [[("a", c)] for c in portions(n, sizes)])["a"]
            assert errors(got, want).max() < 2e-3, (p, sizes)


# -- generation and command -------------------------------------------------------------
def test_greedy_generation(tmp_path):
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    cfg, w, path = _build(tmp_path, "uneven", seed=9)

    def greedy(prompt, n):
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(O.forward(cfg, w, toks)[-1].argmax()))
        return toks[len(prompt):]
    prompts = [tokens_for(cfg, n, 20 + n) for n in (1, 18, 37, 50)]
    prompts.append(prompts[-1][:48] + prompts[0])        # shares full blocks with another
    want = [greedy(p, 12) for p in prompts]
    sp = SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True)
    for kw in (dict(async_scheduling=True), dict(max_num_batched_tokens=16),
               dict(enforce_eager=True), dict(num_gpu_blocks=7, num_cpu_blocks=16)):
        llm = LLM(path, dtype="float32", **{**dict(max_num_seqs=4, max_model_len=128,
                                                   num_gpu_blocks=64), **kw})
        assert [o.outputs[0].token_ids for o in llm.generate(prompts, sp)] == want, kw
        assert [o.outputs[0].token_ids for o in llm.generate(prompts, sp)] == want, kw
    llm = LLM(path, dtype="bfloat16", max_num_seqs=4, max_model_len=128)    # profiled cache size
    outs = llm.generate(prompts, sp)
    assert all(len(o.outputs[0].token_ids) == 12 for o in outs)


def test_trace_run_command(tmp_path):
    cfg, w, path = _build(tmp_path, "wide", seed=3)
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
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32"]
    import numpy as np
    got = np.concatenate([np.fromfile(out / f, dtype="<f4").reshape(-1, cfg["vocab"])
                          for f in ("0.f32", "2.f32")])
    assert errors(torch.from_numpy(got), want[[0, 29, 39]]).max() < 2e-4
    bad = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path],
                         capture_output=True, timeout=120)
    assert bad.returncode != 0
