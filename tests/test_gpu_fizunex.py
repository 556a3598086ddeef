"""Fizunex on the GPU: its kernels against the torch formulation, the engine's step against the
oracle in both dtypes (cache, state slots, portions, mixed batches, CUDA graphs), generation, and the
trace runner as a command."""
import json
import os
import subprocess

import pytest
import torch

import fizunex_oracle as O
from fizunex_cases import (CONFIGS, Step, build, delta, errors, greedy, mixed_steps, model_config,
                           oracle, parallel, portions, replayer, run, tokens_for)

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
    if isinstance(x, tuple):
        return tuple(_cuda(t) for t in x)
    if isinstance(x, dict):
        return {k: _cuda(v) for k, v in x.items()}
    return x.cuda() if torch.is_tensor(x) else x


# -- residual stream and gates ----------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,H", [(3, 72), (2, 37), (300, 2048), (5, 4096), (1, 13000)])
def test_residual_kernels(T, H, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    g = torch.Generator().manual_seed(H)
    wide = torch.randn(T, H + 8, generator=g).to(dtype)
    y = wide[:, :H]
    x, w, b, fw, fb = (torch.randn(*s, generator=g) for s in ((T, H), (H,), (H,), (H,), (H,)))
    gx, glo = C.start_rows(_cuda(wide)[:, :H], 1.7)
    wx, wlo = ref.start_rows(y, 1.7)
    _close(gx, wx, F32)
    _close(glo, wlo, dtype)
    for ln, bias, final in ((True, b, None), (False, None, None), (True, b, fb), (True, None, None)):
        kw = dict(layer_norm=ln, final_weight=fw if final is not None else None, final_bias=final,
                  final_scale=0.4 if final is not None else 1.0)
        out, lo = torch.empty(T, H), torch.empty(T, H)
        ref.add_normed(x, y.float(), w, bias, 1e-4, lo, out=out, **kw)
        gout, glo = _cuda(x).clone(), torch.empty(T, H, dtype=dtype, device="cuda")
        C.add_normed(gout, _cuda(wide)[:, :H], _cuda(w), _cuda(bias), 1e-4, glo, out=gout,
                     **_cuda(kw))
        _close(gout, out, F32)
        _close(glo, lo, dtype)
    u = torch.randn(T, 2 * (H // 2) + 2 * (H % 2), generator=g).to(dtype)
    _close(C.act_mul_rows(u.cuda()), ref.silu_and_mul(u.float()), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,N,V", [(5, 3, 28), (2, 2, 11), (70, 8, 128), (9, 4, 256), (3, 2, 300)])
def test_head_norm_and_gates(T, N, V, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    g = torch.Generator().manual_seed(V)
    o, zw = torch.randn(T, N, V, generator=g) * 3, torch.randn(T, N * V + 16, generator=g).to(dtype)
    w, nq, low = (torch.randn(*s, generator=g) for s in ((N * V,), (T, N), (T, N)))
    z, buf = zw[:, 8:8 + N * V], torch.zeros(T, N * V + 24, dtype=dtype, device="cuda")
    want = torch.empty(T, N * V)
    for wt, a, b in ((w, None, None), (w[:V].clone(), None, None), (w, nq, low.abs())):
        ref.head_norm_gate(o, wt, z.float(), 1e-3, 0.6, want, a, b)
        got = C.head_norm_gate(o.cuda(), wt.cuda(), zw.cuda()[:, 8:8 + N * V], 1e-3, 0.6,
                               buf[:, 8:8 + N * V], _cuda(a), _cuda(b))
        _close(got, want, dtype)
    oc = torch.randn(T, N, V + 4, generator=g).to(dtype)
    ref.head_gate(oc.float(), z.float(), 1.3, V, want)
    _close(C.head_gate(oc.cuda(), zw.cuda()[:, 8:8 + N * V], 1.3, V, buf[:, 8:8 + N * V]), want,
           dtype)
    assert (buf[:, :8] == 0).all() and (buf[:, 8 + N * V:] == 0).all()


# -- attention --------------------------------------------------------------------------
def _paged(Hq, Hkv, D, q_lens, seq_lens, dtype, bs=16, seed=0):
    """Queries that each match one key, far or near, at page and tile edges; the first key the row
    may not see matches best of all."""
    g = torch.Generator().manual_seed(seed)
    B = len(q_lens)
    mb = max(1, -(-max(seq_lens) // bs)) + 1
    nb = B * mb + 3
    kc, vc = torch.randn(nb, bs, Hkv, D, generator=g), torch.randn(nb, bs, Hkv, D, generator=g)
    bt = (torch.randperm(nb - 1, generator=g)[:B * mb] + 1).view(B, mb).int()
    rows = []
    for b, (ql, n) in enumerate(zip(q_lens, seq_lens)):
        for i in range(ql):
            seen = n - ql + i + 1
            for a in range(Hq):
                cand = [c for c in (0, seen - 1, seen // 2, 15, 16, 17, 63, 64, 127, 128, 129)
                        if c < seen]
                if not cand:
                    rows.append(torch.randn(D, generator=g))
                    continue
                p, h = cand[(a + i) % len(cand)], a // (Hq // Hkv)
                k = kc[bt[b, p // bs], p % bs, h]
                row = k * (8.0 * D ** 0.5 / (k @ k))
                if seen < n:
                    f = kc[bt[b, seen // bs], seen % bs, h]
                    row = row + f * (12.0 * D ** 0.5 / (f @ f))
                rows.append(row)
    q = torch.stack(rows).view(sum(q_lens), Hq, D)
    sink = torch.linspace(-2.0, 9.0, Hq)
    cu = torch.tensor([0] + list(torch.tensor(q_lens).cumsum(0)), dtype=torch.int32)
    return (q.to(dtype), kc.to(dtype), vc.to(dtype), bt,
            torch.tensor(seq_lens, dtype=torch.int32), cu, sink)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("Hq,Hkv,D", [(1, 1, 4), (6, 2, 20), (3, 3, 52), (34, 2, 96), (4, 1, 200),
                                      (2, 2, 512)])
def test_general_attention(Hq, Hkv, D, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    ql, sl, nd = [1, 1, 1, 40, 2, 65], [1, 300, 0, 40, 99, 200], 3
    q, kc, vc, bt, s, cu, sink = _paged(Hq, Hkv, D, ql, sl, dtype, bs=8, seed=D)
    scale = D ** -0.5
    rest = (cu[nd:] - cu[nd])
    for sk in (None, sink):
        got = C.any_attention(q.cuda(), kc.cuda(), vc.cuda(), bt.cuda(), s.cuda(), nd, rest.cuda(),
                              scale, _cuda(sk))
        _status()
        _close(got, ref.any_attention(q.float(), kc.float(), vc.float(), bt, s, nd, rest, scale, sk),
               dtype)


@pytest.mark.parametrize("Hq,Hkv,D", [(4, 4, 64), (6, 2, 96), (16, 1, 96), (8, 1, 128), (5, 5, 96)])
def test_tensor_core_attention_with_sinks(Hq, Hkv, D):
    from vllm_gcu_b200.ops import cuda as C, ref
    scale = D ** -0.5
    ql, sl = [40, 7, 130, 1, 256], [40, 300, 130, 9, 700]
    q, kc, vc, bt, s, cu, sink = _paged(Hq, Hkv, D, ql, sl, BF16, seed=D)
    for sk in (None, sink):
        got = C.fmha_prefill_sink(q.cuda(), kc.cuda(), vc.cuda(), bt.cuda(), cu.cuda(), s.cuda(),
                                  scale, sum(-(-n // 128) for n in ql), _cuda(sk))
        _status()
        _close(got, ref.any_attention(q.float(), kc.float(), vc.float(), bt, s, 0, cu, scale, sk),
               BF16)
    sl = [1, 17, 64, 65, 600, 0]
    q, kc, vc, bt, s, cu, sink = _paged(Hq, Hkv, D, [1] * 6, sl, BF16, seed=D + 1)
    want = ref.any_attention(q.float(), kc.float(), vc.float(), bt, s, 6, None, scale, sink)
    for splits in (1, 3):
        got = C.paged_decode(q.cuda(), kc.cuda(), vc.cuda(), bt.cuda(), s.cuda(), scale,
                             num_splits=splits, sink=sink.cuda())
        _status()
        _close(got, want, BF16)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("Hq,Hkv,D,DC,rot", [(6, 2, 20, 64, 12), (3, 3, 7, 64, 4), (8, 4, 96, 96, 32),
                                             (32, 8, 128, 128, 64), (5, 1, 40, 64, 40),
                                             (2, 1, 30, 64, 0), (64, 8, 128, 128, 128),
                                             (80, 80, 128, 128, 8)])
def test_key_norm_rotation_and_cache(Hq, Hkv, D, DC, rot, dtype):
    from vllm_gcu_b200.layers.basic import build_cos_sin_cache
    from vllm_gcu_b200.ops import cuda as C, ref
    g = torch.Generator().manual_seed(D)
    T, nb, bs = 9, 5, 4
    wide = (3 * torch.randn(T, (Hq + 2 * Hkv) * D + 8, generator=g)).to(dtype)
    cut = lambda t: (t[:, :Hq * D], t[:, Hq * D:(Hq + Hkv) * D],  # noqa: E731
                     t[:, (Hq + Hkv) * D:(Hq + 2 * Hkv) * D])
    qw, kw = 1 + torch.rand(Hq * D, generator=g), torch.randn(Hkv * D, generator=g)
    cs = build_cos_sin_cache(rot, 50, 500.0, None)
    pos = torch.randint(0, 50, (T,), generator=g)
    slots = torch.randperm(nb * bs, generator=g)[:T]
    slots[3] = -1
    for own_v, neox, ss in ((False, False, None), (True, False, None), (False, rot > 0, None),
                            (False, False, 4 * torch.rand(T, 2, generator=g) * D)):
        caches = [torch.full((nb, bs, Hkv, DC), 2.0).to(dtype) for _ in range(2)]
        dev = [c.cuda() for c in caches]
        q, k, v = cut(wide)
        want = ref.qk_norm_rope_cache(q, k, v if own_v else None, qw, kw, 1e-4, cs, neox, pos, slots,
                                      *caches, D, ss, 2 if ss is not None else 1)
        q, k, v = cut(wide.cuda())
        got = C.qk_norm_rope_cache(q, k, v if own_v else None, qw.cuda(), kw.cuda(), 1e-4, cs.cuda(),
                                   neox, pos.cuda(), slots.cuda(), *dev, D, _cuda(ss),
                                   2 if ss is not None else 1)
        _status()
        _close(got, want, dtype)
        for a, b in zip(dev, caches):
            _close(a, b, dtype)


# -- recurrences ------------------------------------------------------------------------
# (slot, first position, tokens): single tokens first, a fresh one among them, one without a slot
STEP = [(3, 0, 1), (0, 37, 1), (-1, 5, 1), (6, 1, 1), (2, 0, 40), (5, 9, 2), (1, 2, 17), (4, 0, 3),
        (7, 100, 33)]


def _delta_case(N, G, D, V, taps, step, dtype, seed):
    from vllm_gcu_b200.layers.recurrent import state_rows
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    rows, C_ = state_rows(D, "t"), 2 * G * D + N * V
    pad = (-C_) % 8
    wide = r(step.T, C_ + pad + 8).to(dtype)
    kw = dict(z=r(step.T, N * D) - 1, b=r(step.T, N),
              conv=tuple(0.7 * r(taps, n) for n in (G * D, G * D, N * V)), dt_bias=r(N * D),
              a_log=r(N))
    state = {"matrix": torch.zeros(8, N, V, rows), "taps": r(8, taps, C_).to(dtype)}
    state["matrix"][..., :D] = r(8, N, V, D)
    cut = lambda t: (t[:, :G * D], t[:, G * D:2 * G * D], t[:, 2 * G * D:C_])  # noqa: E731
    return wide, cut, kw, state, rows


DELTA_SIZES = [(6, 3, 20, 28, 3), (3, 1, 5, 7, 5), (2, 2, 32, 32, 1), (2, 1, 64, 48, 2),
               (4, 4, 96, 160, 4), (40, 40, 128, 128, 4), (2, 1, 136, 40, 7), (2, 2, 256, 300, 8),
               (70, 35, 48, 64, 3), (64, 64, 8, 12, 4), (40, 20, 200, 72, 3)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("N,G,D,V,taps", DELTA_SIZES)
def test_gated_delta_rule(N, G, D, V, taps, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    step = Step(STEP, pad=2)
    wide, cut, kw, state, rows = _delta_case(N, G, D, V, taps, step, dtype, N + D)
    dstate = _cuda({k: v.clone() for k, v in state.items()})
    n = step.T - 2
    want = ref.delta_rule(*cut(wide), **kw, head_dim=D, v_dim=V, rows=rows, md=step, state=state)
    got = C.delta_rule(*cut(wide.cuda()), **_cuda(kw), head_dim=D, v_dim=V, rows=rows,
                       md=step.to("cuda"), state=dstate)
    _status()
    lim = F32 if dtype == F32 else BF16          # (fast exponentials: far below a bf16 rounding)
    scale = max(1.0, want[:n].abs().max().item()) * (3 if dtype == F32 else 0.05)
    _close(got[:n], want[:n], lim, scale)
    _close(dstate["matrix"], state["matrix"], lim, max(1.0, state["matrix"].abs().max().item())
           * (3 if dtype == F32 else 0.05))
    assert torch.equal(dstate["taps"].cpu(), state["taps"])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("N,G,D,V,taps", DELTA_SIZES)
def test_gated_delta_single_tokens(N, G, D, V, taps, dtype):
    """The fused step against scan, norm and gate."""
    from vllm_gcu_b200.ops import cuda as C, ref
    H = 72 if N != 3 else 37
    step = Step([(3, 0, 1), (0, 37, 1), (-1, 5, 1), (6, 1, 1), (7, 1000, 1), (1, 2, 1)])
    wide, cut, kw, state, rows = _delta_case(N, G, D, V, taps, step, dtype, N + D)
    g = torch.Generator().manual_seed(1)
    h, wb = torch.randn(step.T, H, generator=g).to(dtype), torch.randn(N, H, generator=g).to(dtype)
    gate = torch.randn(step.T, N * V, generator=g).to(dtype)
    norm = torch.randn(V, generator=g)
    kw["b"] = h.float() @ wb.float().T
    dstate = _cuda({k: v.clone() for k, v in state.items()})
    o = ref.delta_rule(*cut(wide), **kw, head_dim=D, v_dim=V, rows=rows, md=step, state=state)
    want = torch.zeros(step.T, N * V)
    ref.head_norm_gate(o, norm, gate.float(), 1e-4, 0.8, want)
    out = torch.full((step.T, N * V + 8), 9.0, dtype=dtype, device="cuda")
    d = _cuda(kw)
    C.delta_step(h.cuda(), *cut(wide.cuda()), d["z"], gate.cuda(), wb.cuda(), d["conv"],
                 d["dt_bias"], d["a_log"], norm.cuda(), D, V, rows, step.positions.cuda(),
                 step.state_slots.cuda(), dstate, 1e-4, 0.8, out[:, :N * V])
    _status()
    want[2] = 0                                   # no slot: zeros
    _close(out[:, :N * V], want, dtype, 3 * max(1.0, want.abs().max().item()))
    assert (out[:, N * V:] == 9).all()
    _close(dstate["matrix"], state["matrix"], F32 if dtype == F32 else BF16,
           max(1.0, state["matrix"].abs().max().item()) * (3 if dtype == F32 else 0.05))
    assert torch.equal(dstate["taps"].cpu(), state["taps"])


MEMORY_SIZES = [(3, 12, 20, 9.0), (2, 3, 11, 4.0), (1, 32, 4, 1.0), (2, 160, 48, 12.0),
                (4, 64, 64, 15.0), (9, 128, 256, 15.0), (80, 96, 63, 6.0), (2, 200, 260, 10.0),
                (64, 128, 127, 15.0), (48, 256, 40, 8.0)]


def _memory_case(N, D, V, step, dtype):
    from vllm_gcu_b200.layers.recurrent import state_rows
    g = torch.Generator().manual_seed(N + D)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    rows, width = state_rows(D, "t"), N * (2 * D + 2 * V)
    wide = r(step.T, width + (-width) % 8).to(dtype)
    cut = lambda t: t[:, :width].split([N * D, N * D, N * V, N * V], dim=1)  # noqa: E731
    state = {"matrix": torch.zeros(8, N, V, rows), "vector": torch.zeros(8, N, rows),
             "scalar": r(8, N)}
    state["matrix"][..., :D], state["vector"][..., :D] = r(8, N, V, D), r(8, N, D)
    return wide, cut, state, rows, r


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("N,D,V,cap", MEMORY_SIZES)
def test_matrix_memory(N, D, V, cap, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    step = Step(STEP, pad=2)
    wide, cut, state, rows, r = _memory_case(N, D, V, step, dtype)
    gates = (4 * r(step.T, N), 4 * r(step.T, N) + 3, r(N), r(N))
    dstate = _cuda({k: v.clone() for k, v in state.items()})
    n = step.T - 2
    args = dict(cap=cap, head_dim=D, v_dim=V, rows=rows)
    o, nq, low = ref.matrix_memory(*cut(wide)[:3], *gates, **args, md=step, state=state)
    go, gnq, glow = C.matrix_memory(*cut(wide.cuda())[:3], *_cuda(gates), **args,
                                    md=step.to("cuda"), state=dstate)
    _status()
    low[2] = 1.0
    for a, b in ((go[:n], o[:n]), (gnq[:n], nq[:n]), (glow[:n], low[:n]),
                 *((dstate[k], state[k]) for k in state)):
        _close(a, b, F32, 3 * max(1.0, b.abs().max().item()))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("N,D,V,cap", MEMORY_SIZES)
def test_matrix_memory_single_tokens(N, D, V, cap, dtype):
    from vllm_gcu_b200.ops import cuda as C, ref
    H = 72 if N != 2 else 37
    step = Step([(3, 0, 1), (0, 37, 1), (-1, 5, 1), (6, 1, 1), (7, 1000, 1), (1, 2, 1)])
    wide, cut, state, rows, r = _memory_case(N, D, V, step, dtype)
    h, wi, wf = (r(*s).to(dtype) for s in ((step.T, H), (N, H), (N, H)))
    ib, fb, norm = r(N), r(N) + 3, r(N * V)
    dstate = _cuda({k: v.clone() for k, v in state.items()})
    q, k, v, gate = cut(wide)
    o, nq, low = ref.matrix_memory(q, k, v, h.float() @ wi.float().T, h.float() @ wf.float().T, ib,
                                   fb, cap, D, V, rows, step, state)
    want = torch.zeros(step.T, N * V)
    ref.head_norm_gate(o, norm, gate.float(), 1e-4, 0.8, want, nq, low)
    want[2] = 0
    out = torch.empty(step.T, N * V, dtype=dtype, device="cuda")
    q, k, v, gate = cut(wide.cuda())
    C.memory_step(h.cuda(), q, k, v, gate, wi.cuda(), wf.cuda(), ib.cuda(), fb.cuda(), cap,
                  norm.cuda(), D, V, rows, step.positions.cuda(), step.state_slots.cuda(), dstate,
                  1e-4, 0.8, out)
    _status()
    _close(out, want, dtype, 3 * max(1.0, want.abs().max().item()))
    for key in state:
        _close(dstate[key], state[key], F32, 3 * max(1.0, state[key].abs().max().item()))


# -- the engine's step ------------------------------------------------------------------
GPU_CONFIGS = {**CONFIGS,
               # more query heads per key head than the decode kernel takes, heads wider than the
               # tensor-core kernels', states of the largest sizes
               "big": model_config(120, 128, [
                   parallel((34, 2, 40, 16, 1e4, 0.15), (2, 200, 260, 10.0), ff=64),
                   delta(2, 1, 256, 300, 8, 32),
                   parallel((4, 2, 144, 48, 1e5, 0.09), (4, 64, 64, 15.0)),
                   parallel((4, 1, 128, 128, 1e6, 0.09), (1, 128, 128, 15.0)),
                   delta(4, 4, 64, 64, 4)]),
               "even": model_config(256, 256, [delta(4, 4, 64, 64, 4, 256),
                                               parallel((4, 2, 64, 32, 1e4, 0.125),
                                                        (2, 64, 128, 15.0), ff=256)])}


def _check(got, want, dtype, what=""):
    e = errors(got, want)
    if dtype == "float32":
        assert e.max() < 5e-4, (what, e.max())
    else:
        # rounding, and a few rows at which a normaliser is close to nothing
        assert (e > 0.08).float().mean() <= 0.04 or int((e > 0.08).sum()) <= 1, (what, e)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(GPU_CONFIGS))
def test_portions_and_decoding(tmp_path, name, dtype):
    cfg, w, path = build(tmp_path, name, configs=GPU_CONFIGS)
    toks = tokens_for(cfg, 150)
    want = oracle(cfg, w, {"a": toks})["a"]
    rp = replayer(path, "cuda", dtype, max_tokens=192)
    for sizes in ([150], [2, 3, 64, 1], [31, 2, 1], [100] + [1] * 50):
        got = run(rp, {"a": toks}, [[("a", n)] for n in portions(150, sizes)])["a"]
        _check(got, want, dtype, sizes)
    assert rp.engine.runner.graph_launches > 0           # decoded through CUDA graphs
    _status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["uneven", "wide"])
def test_mixed_batches_and_reused_slots(tmp_path, name, dtype):
    cfg, w, path = build(tmp_path, name, seed=5)
    prompts = {f"r{i}": tokens_for(cfg, n, i) for i, n in
               enumerate((1, 40, 2, 65, 17, 130, 33, 3, 64, 16))}
    want = oracle(cfg, w, prompts)
    rp = replayer(path, "cuda", dtype, max_tokens=384)
    got = run(rp, prompts, mixed_steps(prompts))
    for k in prompts:
        _check(got[k], want[k], dtype, k)
    kv = rp.engine.scheduler.kv
    assert kv.pool.num_free_blocks == kv.pool.num_blocks and len(kv.free_slots) == 4


def test_far_tokens(tmp_path):
    cfg, w, path = build(tmp_path, "uneven", seed=4, far=3.0)
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
    cfg, w, path = build(tmp_path, "uneven", seed=9)
    prompts = [tokens_for(cfg, n, 20 + n) for n in (1, 18, 37, 50)]
    prompts.append(prompts[-1][:48] + prompts[0])        # shares full blocks with another
    want = [greedy(cfg, w, p, 12) for p in prompts]
    sp = SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True)
    for kw in (dict(async_scheduling=True), dict(max_num_batched_tokens=16),
               dict(enforce_eager=True), dict(num_gpu_blocks=7)):
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
    assert errors(torch.from_numpy(got), want[[0, 29, 39]]).max() < 5e-4
