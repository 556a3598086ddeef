"""Fizunex on the CPU path: every mechanism against the oracle's equations, then the engine's step
(cache, state slots, batches, portions) and its generation path against whole-sequence evaluation."""
import math

import pytest
import torch

import fizunex_oracle as O
from fizunex_cases import (CONFIGS, Step, build, delta, errors, greedy, mixed_steps, model_config,
                           oracle, parallel, portions, replayer, run, spread, tokens_for,
                           write_checkpoint)

TOL = 5e-5


def gen(seed):
    return torch.Generator().manual_seed(seed)


# -- mechanisms -------------------------------------------------------------------------
def test_start_rows_and_added_norms():
    from vllm_gcu_b200.ops import ref
    g = gen(0)
    T, H = 5, 14
    e, y, w, b, fw, fb = (torch.randn(*s, generator=g) for s in
                          ((T, H), (T, H), (H,), (H,), (H,), (H,)))
    x, lo = ref.start_rows(e, 2.5)
    assert torch.allclose(x, e * 2.5) and torch.allclose(lo, x)
    want = x + O.layer_norm(y, w, b, 1e-3)
    out, lo = torch.empty(T, H), torch.empty(T, H)
    ref.add_normed(x, y, w, b, 1e-3, lo, out=out)
    assert torch.allclose(out, want, atol=1e-5) and torch.equal(lo, out)
    ref.add_normed(x, y, w, b, 1e-3, lo, final_weight=fw, final_bias=fb, final_scale=0.3)
    assert torch.allclose(lo, O.layer_norm(want, fw, fb, 1e-3) * 0.3, atol=1e-5)
    ref.add_normed(x, y, w, None, 1e-3, lo, layer_norm=False)
    assert torch.allclose(lo, x + O.rms_unit(y, 1e-3) * w, atol=1e-5)


@pytest.mark.parametrize("heads,kv,dim,rot", [(6, 2, 8, 4), (3, 3, 5, 4), (1, 1, 6, 6), (4, 1, 12, 0)])
def test_key_attention_layer(heads, kv, dim, rot):
    """Norm over the whole projection, pairs of neighbours rotated, values taken before both, one
    sink per head, the gate; a whole prompt and then single tokens over a paged cache."""
    from vllm_gcu_b200.config import AttentionSpec
    from vllm_gcu_b200.layers.attention import AttentionMetadata
    from vllm_gcu_b200.layers.basic import RotaryEmbedding
    from vllm_gcu_b200.layers.key_attention import KeyAttention
    from vllm_gcu_b200.layers.mixer import MixerBlock
    g = gen(heads)
    H, T, bs, eps = 20, 13, 4, 1e-3
    spec = AttentionSpec(heads, kv, dim, 0.45, rot, 30.0)
    part = KeyAttention(spec, eps, torch.float32, "cpu", "p",
                        RotaryEmbedding(dim, rot, 64, 30.0, is_neox=False, keep_fp32=True))
    m = MixerBlock([("", 1.0, part)], H, torch.float32, "cpu", "p")
    q, k = heads * dim, kv * dim
    w = {n: torch.randn(*s, generator=g) * s[-1] ** -0.5 for n, s in
         {"q": (q, H), "k": (k, H), "g": (q, H), "o": (H, q)}.items()}
    w.update({"q.norm": 2 + torch.rand(q, generator=g), "k.norm": 1 + torch.rand(k, generator=g),
              "sink": torch.randn(heads, generator=g)})
    assert m.tensor_names() == set(w) and all(m.load(n, t) for n, t in w.items())
    h = torch.randn(T, H, generator=g)
    want = O.key_value_attention(h.double(), {n: t.double() for n, t in w.items()}, heads, kv, dim,
                                 rot, 30.0, 0.45, eps)
    cache = torch.full((2, 6, bs, *part.cache_shape()), 7.0)
    bt = torch.tensor([[4, 1, 3, 0]], dtype=torch.int32)
    got, at = [], 0
    for n in (9, 1, 1, 2):
        pos = torch.arange(at, at + n)
        md = AttentionMetadata(
            num_tokens=n, num_decodes=int(n == 1), num_prefills=int(n > 1),
            num_decode_tokens=int(n == 1), positions=pos, block_tables=bt,
            slot_mapping=bt[0][pos // bs].long() * bs + pos % bs,
            seq_lens=torch.tensor([at + n], dtype=torch.int32),
            cu_q_prefill=torch.tensor([0, n], dtype=torch.int32) if n > 1 else None)
        got.append(m(h[at:at + n], md, cache, None))
        at += n
    assert torch.allclose(torch.cat(got).double(), want, atol=1e-5)
    # the sink matters, and its size does
    w["sink"] = w["sink"] - 3
    other = O.key_value_attention(h, w, heads, kv, dim, rot, 30.0, 0.45, eps)
    assert (other - want).abs().max() > 1e-2


SCHEDULES = [[(0, 11)], [(0, 1)] * 11, [(0, 2), (0, 3), (0, 1), (0, 5)], [(0, 8), (0, 2), (0, 1)]]


def _delta_inputs(N, G, D, V, taps, T, seed):
    g = gen(seed)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    return dict(q=r(T, G * D), k=r(T, G * D), v=r(T, N * V), z=r(T, N * D) - 1, b=r(T, N),
                conv=tuple(0.7 * r(taps, n) for n in (G * D, G * D, N * V)),
                dt_bias=r(N * D), a_log=r(N))


def _delta_want(x, N, G, D, V):
    d = {k: (tuple(t.double() for t in v) if isinstance(v, tuple) else v.double())
         for k, v in x.items()}
    T = d["q"].shape[0]
    q, k, v = (O.silu(O.short_conv(d[c], t.T)) for c, t in zip("qkv", d["conv"]))
    step = O.softplus(d["z"] + d["dt_bias"]).view(T, N, D)
    return O.delta_rule(O.unit(q.view(T, G, D)) * D ** -0.5, O.unit(k.view(T, G, D)),
                        v.view(T, N, V), torch.exp(-torch.exp(d["a_log"])[None, :, None] * step),
                        O.sigmoid(d["b"]))


@pytest.mark.parametrize("N,G,D,V,taps", [(4, 2, 6, 5, 3), (1, 1, 3, 7, 1), (3, 3, 8, 4, 6)])
def test_gated_delta_rule_portions_and_slots(N, G, D, V, taps):
    from vllm_gcu_b200.layers.recurrent import state_rows
    from vllm_gcu_b200.ops import ref
    x = _delta_inputs(N, G, D, V, taps, 11, 1)
    want = _delta_want(x, N, G, D, V)
    rows = state_rows(D, "t")
    C = 2 * G * D + N * V
    state = {"matrix": torch.full((3, N, V, rows), 5.0), "taps": torch.full((3, taps, C), -4.0)}
    for sch in SCHEDULES:                       # each leaves its state behind in the slot
        at, got = 0, []
        for slot, n in sch:
            s = slice(at, at + n)
            step = Step([(slot, at, n)], decodes=int(n == 1 and at % 2 == 0))
            got.append(ref.delta_rule(x["q"][s], x["k"][s], x["v"][s], x["z"][s], x["b"][s],
                                      x["conv"], x["dt_bias"], x["a_log"], D, V, rows, step, state))
            at += n
        assert torch.allclose(torch.cat(got).double(), want, atol=1e-5), sch
    assert (state["matrix"][1:] == 5.0).all()   # other slots are left alone


@pytest.mark.parametrize("N,D,V,cap", [(3, 4, 6, 5.0), (1, 7, 2, 1.0), (2, 5, 5, 15.0)])
def test_matrix_memory_portions_and_slots(N, D, V, cap):
    from vllm_gcu_b200.layers.recurrent import state_rows
    from vllm_gcu_b200.ops import ref
    g = gen(N)
    T = 11
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    q, k, v, zi, zf = r(T, N * D), r(T, N * D), r(T, N * V), 4 * r(T, N), 4 * r(T, N) + 3
    ib, fb = r(N), r(N)
    i, f = O.memory_gates((zi + ib).double(), (zf + fb).double(), cap)
    want = O.matrix_memory(q.double().view(T, N, D) * D ** -0.5, k.double().view(T, N, D),
                           v.double().view(T, N, V), i, f)
    rows = state_rows(D, "t")
    state = {"matrix": torch.full((2, N, V, rows), 5.0), "vector": torch.full((2, N, rows), 5.0),
             "scalar": torch.full((2, N), 5.0)}
    for sch in SCHEDULES:
        at, got = 0, []
        for slot, n in sch:
            s = slice(at, at + n)
            o, nq, low = ref.matrix_memory(q[s], k[s], v[s], zi[s], zf[s], ib, fb, cap, D, V, rows,
                                           Step([(slot, at, n)], decodes=0), state)
            got.append(o / (torch.maximum(nq.abs(), low) + 1e-6).unsqueeze(-1))
            at += n
        assert torch.allclose(torch.cat(got).double(), want, rtol=1e-4, atol=1e-5), sch


def test_head_norm_and_gates():
    from vllm_gcu_b200.ops import ref
    g = gen(3)
    T, N, V = 4, 3, 6
    o, z, w = torch.randn(T, N, V, generator=g), torch.randn(T, N * V, generator=g), \
        torch.randn(N * V, generator=g)
    out = torch.empty(T, N * V)
    ref.head_norm_gate(o, w, z, 1e-2, 0.7, out)
    want = O.rms_unit(o, 1e-2).reshape(T, N * V) * w * O.sigmoid(z) * 0.7
    assert torch.allclose(out, want, atol=1e-6)
    ref.head_norm_gate(o, w[:V], z, 1e-2, 1.0, out)
    want = (O.rms_unit(o, 1e-2) * w[:V]).reshape(T, N * V) * O.sigmoid(z)
    assert torch.allclose(out, want, atol=1e-6)
    ref.head_gate(o, z[:, :N * 4], 0.5, 4, out[:, :N * 4])
    assert torch.allclose(out[:, :N * 4], o[..., :4].reshape(T, -1) * O.sigmoid(z[:, :N * 4]) * 0.5)


# -- configuration ----------------------------------------------------------------------
def test_configuration_reads_every_number():
    from vllm_gcu_b200.config import AttentionSpec, DeltaSpec, MemorySpec, ModelConfig
    cfg = ModelConfig.from_hf_dict(CONFIGS["uneven"], dtype="float32")
    assert (cfg.embed_scale, cfg.logit_scale, cfg.rms_norm_eps) == (1.7, 0.6, 1e-4)
    (n0, s0, d0), = cfg.layer_specs[0].parts
    assert d0 == DeltaSpec(6, 3, 20, 28, 3, 20, 20) and (n0, s0) == ("", 1.0)
    left, right = cfg.layer_specs[1].parts
    assert left == ("left.", 0.8, AttentionSpec(6, 2, 20, 0.3, 12, 1000.0))
    assert right == ("right.", 1.3, MemorySpec(3, 12, 20, 9.0))
    assert [s.has_mlp for s in cfg.layer_specs] == [True, True, False, False]
    assert cfg.kv_bytes_per_token() == 4 * 2 * (2 * 20 + 4 * 16)
    bad = model_config(8, 8, [parallel((2, 1, 4, 2, 10.0, 1.0), (1, 2, 2, 1.0))])
    bad["layers"][0]["mixer"]["left"]["vdim"] = 8
    with pytest.raises(ValueError, match="values are the keys"):
        ModelConfig.from_hf_dict(bad)
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        ModelConfig.from_hf_dict(bad)


def test_ranks_come_from_the_checkpoint(tmp_path):
    from vllm_gcu_b200.config import ModelConfig
    cfg = CONFIGS["uneven"]
    path = write_checkpoint(tmp_path / "m", cfg, O.random_model(cfg, 0, ranks=(11, 3)))
    mc = ModelConfig.from_pretrained(path)
    spec = mc.layer_specs[2].parts[0][2]
    assert (spec.decay_rank, spec.gate_rank) == (11, 3)
    toks = tokens_for(cfg, 20)
    got = run(replayer(path, "cpu", max_tokens=64), {"a": toks}, [[("a", 20)]])["a"]
    w = O.random_model(cfg, 0, ranks=(11, 3))
    assert errors(got, O.forward(cfg, w, toks)).max() < TOL


def test_missing_tensors_and_bad_sizes_are_refused(tmp_path):
    from vllm_gcu_b200.config import ModelConfig
    from vllm_gcu_b200.models import build_model
    cfg = CONFIGS["ones"]
    w = O.random_model(cfg, 0)
    m = build_model(ModelConfig.from_hf_dict(
        cfg, dtype="float32", tensor_shapes={k: tuple(v.shape) for k, v in w.items()}), "cpu")
    del w["l0.mix.left.sink"]
    with pytest.raises(ValueError, match="missing"):
        m.load_weights(w.items())
    for layer, msg in ((delta(2, 1, 300, 4, 2), "keys per head"), (delta(2, 1, 4, 4, 9), "taps"),
                       (delta(3, 2, 4, 4, 2), "heads"),
                       (parallel((2, 1, 6, 3, 10.0, 1.0), (1, 2, 2, 1.0)), "rotated")):
        with pytest.raises(ValueError, match=msg):
            build_model(ModelConfig.from_hf_dict(model_config(8, 8, [layer]), dtype="float32"), "cpu")


# -- the engine's step ------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_portions_and_decoding_match_the_oracle(tmp_path, name):
    cfg, w, path = build(tmp_path, name)
    toks = tokens_for(cfg, 53)
    want = oracle(cfg, w, {"a": toks})["a"]
    rp = replayer(path, "cpu", max_tokens=128)
    for sizes in ([53], [1], [2], [3, 2, 7], [16, 1], [31, 2, 1], [17, 15, 16]):
        got = run(rp, {"a": toks}, [[("a", n)] for n in portions(53, sizes)])["a"]
        assert errors(got, want).max() < TOL, sizes


def test_far_tokens_count_at_page_borders_and_at_the_start(tmp_path):
    """Swapping one token at a far position, at the edges of pages and at the start changes late
    logits, and the engine follows the oracle either way, in a prompt and in decoding."""
    cfg, w, path = build(tmp_path, "uneven", seed=4, far=3.0)
    n = 150
    base = tokens_for(cfg, n, 7)
    rp = replayer(path, "cpu", max_tokens=256)
    before = O.forward(cfg, w, base)
    moved = 0
    for p in (0, 1, 15, 16, 17, 31, 32, 64, 127):
        toks = list(base)
        toks[p] = (toks[p] + 1) % cfg["vocab"]
        want = O.forward(cfg, w, toks)
        moved += int((errors(want, before)[-20:] > 3e-3).any())
        for sizes in ([n], [n - 6, 1, 1, 1, 1, 1, 1]):
            got = run(rp, {"a": toks}, [[("a", c)] for c in portions(n, sizes)])["a"]
            assert errors(got, want).max() < 1e-3, (p, sizes)
    assert moved >= 7


def test_batches_match_each_request_alone_and_slots_are_used_again(tmp_path):
    cfg, w, path = build(tmp_path, "uneven", seed=5)
    prompts = {f"r{i}": tokens_for(cfg, n, i) for i, n in
               enumerate((1, 40, 2, 65, 17, 70, 33, 3, 64, 16))}
    want = oracle(cfg, w, prompts)
    rp = replayer(path, "cpu", max_tokens=320)      # room for about four requests
    kv = rp.engine.scheduler.kv
    slots = []
    real = kv.allocate_slots

    def allocate(req, *a, **k):
        new = req.state_slot < 0
        out = real(req, *a, **k)
        if new:
            slots.append(req.state_slot)
        return out
    kv.allocate_slots = allocate
    steps = mixed_steps(prompts)
    assert max(len(s) for s in steps) >= 3
    got = run(rp, prompts, steps)
    for k in prompts:
        assert errors(got[k], want[k]).max() < TOL, k
    assert len(slots) == 10 and set(slots) <= {0, 1, 2, 3} and sorted(kv.free_slots) == [0, 1, 2, 3]
    assert kv.pool.num_free_blocks == 20 and not rp.live


def test_a_request_can_pause_while_others_run(tmp_path):
    cfg, w, path = build(tmp_path, "prime", seed=6)
    prompts = {"a": tokens_for(cfg, 40, 1), "b": tokens_for(cfg, 47, 2)}
    want = oracle(cfg, w, prompts)
    rp = replayer(path, "cpu", max_tokens=128)
    steps = [[("a", 17)], [("b", 15)], [("b", 2)], [("b", 1)], [("a", 1)], [("b", 14), ("a", 2)],
             [("b", 15)], [("a", 20)]]
    got = run(rp, prompts, steps)
    assert all(errors(got[k], want[k]).max() < TOL for k in prompts)


def test_long_decoding(tmp_path):
    cfg, w, path = build(tmp_path, "ones", seed=7)
    prompts = {"a": tokens_for(cfg, 210, 1), "b": tokens_for(cfg, 190, 2)}
    want = oracle(cfg, w, prompts)
    rp = replayer(path, "cpu", max_tokens=512)
    steps = spread([("a", 2)] + [("a", 1)] * 208, [("b", 1)] * 190)
    got = run(rp, prompts, steps)
    assert all(errors(got[k], want[k]).max() < TOL for k in prompts)


def test_a_planted_mistake_shows(tmp_path):
    """The comparison is sharp enough: oracles with one mistake each are told apart from the
    engine."""
    cfg, w, path = build(tmp_path, "uneven", seed=8)
    toks = tokens_for(cfg, 30)
    got = run(replayer(path, "cpu", max_tokens=64), {"a": toks}, [[("a", 30)]])["a"]
    assert errors(got, O.forward(cfg, w, toks)).max() < TOL
    real = {n: getattr(O, n) for n in ("sink_softmax", "matrix_memory", "delta_rule", "short_conv",
                                       "rotate_pairs", "memory_gates")}
    conv = real["short_conv"]
    wrong = {
        "sink_softmax": lambda s, sink: torch.softmax(s, -1),
        "matrix_memory": lambda q, k, v, i, f: real["matrix_memory"](
            q, k, v, i, torch.cat([f[:9], f[9:10] - 50, f[10:]])),            # a lost state
        "delta_rule": lambda q, k, v, g, b: real["delta_rule"](
            q, k, v, torch.cat([g[:9], 0 * g[9:10], g[10:]]), b),
        "short_conv": lambda x, t: torch.cat([conv(x[:16], t), conv(x[16:], t)]),
        "rotate_pairs": lambda x, d, b: torch.cat([real["rotate_pairs"](x, d, b)[:-1], x[-1:]]),
        "memory_gates": lambda zi, zf, cap: (zi, real["memory_gates"](zi, zf, cap)[1]),
    }
    for name, f in wrong.items():
        setattr(O, name, f)
        try:
            assert errors(got, O.forward(cfg, w, toks)).max() > 50 * TOL, name
        finally:
            setattr(O, name, real[name])


# -- generation -------------------------------------------------------------------------
@pytest.mark.parametrize("kw", [
    dict(), dict(async_scheduling=True), dict(max_num_batched_tokens=16, max_num_seqs=3),
    dict(num_gpu_blocks=7, num_cpu_blocks=32), dict(num_scheduler_steps=3)],
    ids=["plain", "async", "chunked", "preempt", "multistep"])
def test_greedy_generation_through_the_engine(tmp_path, kw):
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    cfg, w, path = build(tmp_path, "uneven", seed=9)
    prompts = [tokens_for(cfg, n, 20 + n) for n in (1, 18, 37, 16, 50)]
    prompts.append(prompts[-1][:48] + prompts[0])        # shares full blocks with another
    llm = LLM(path, device="cpu", dtype="float32", **{
        **dict(max_num_seqs=4, max_model_len=128, num_gpu_blocks=64), **kw})
    want = [greedy(cfg, w, p, 10) for p in prompts]
    sp = SamplingParams(max_tokens=10, temperature=0.0, ignore_eos=True)
    for _ in range(2):                                   # slots and blocks of the first pass again
        outs = llm.generate(prompts, sp)
        assert [o.outputs[0].token_ids for o in outs] == want
        assert all(o.num_cached_tokens == 0 for o in outs)
    sch = llm.engine.scheduler
    if kw.get("num_gpu_blocks") == 7:
        assert sch.num_preemptions > 0 and sch.num_swaps == 0
    assert len(sch.kv.free_slots) == llm.engine.cfg.scheduler.max_num_seqs


def test_sampling_and_logprobs(tmp_path):
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    cfg, w, path = build(tmp_path, "ones", seed=11)
    llm = LLM(path, device="cpu", dtype="float32", max_num_seqs=4, max_model_len=64)
    p = tokens_for(cfg, 9)
    a, b = (llm.generate([p], SamplingParams(max_tokens=6, temperature=0.8, seed=3, ignore_eos=True))
            for _ in range(2))
    assert a[0].outputs[0].token_ids == b[0].outputs[0].token_ids
    o = llm.generate([p], SamplingParams(max_tokens=1, temperature=0.0, logprobs=2,
                                         prompt_logprobs=0, ignore_eos=True))[0]
    lp = torch.log_softmax(O.forward(cfg, w, p), -1)
    t = o.outputs[0].token_ids[0]
    assert math.isclose(o.outputs[0].logprobs[0][t], float(lp[-1, t]), abs_tol=1e-4)
    for i in range(1, 9):
        assert math.isclose(o.prompt_logprobs[i][p[i]], float(lp[i - 1, p[i]]), abs_tol=1e-4)


def test_what_a_recurrent_state_rules_out(tmp_path):
    from vllm_gcu_b200.config import EngineConfig, ModelConfig, SpeculativeConfig
    from vllm_gcu_b200.engine.llm import LLMEngine
    cfg, w, path = build(tmp_path, "ones")
    mc = ModelConfig.from_pretrained(path, dtype="float32")
    with pytest.raises(ValueError, match="draft tokens"):
        LLMEngine(EngineConfig(model=mc, device="cpu", load_format="safetensors", model_path=path,
                               speculative=SpeculativeConfig("ngram", 2)))
    eng = LLMEngine(EngineConfig(model=mc, device="cpu", load_format="safetensors",
                                 model_path=path))
    assert not eng.scheduler.kv.pool.enable_prefix_caching and not eng.scheduler.cpu_free
    with pytest.raises(ValueError, match="does not ship"):
        eng.attach_kv_connector(object())


def test_presets_and_native_sources():
    from vllm_gcu_b200.config import preset
    from vllm_gcu_b200.csrc import build as b
    from vllm_gcu_b200.models import build_model
    from vllm_gcu_b200.models.fizunex import FizunexForCausalLM
    m = build_model(preset("tiny-fizunex", dtype="float32"), "cpu")
    m.init_random(0)
    assert [s is None for s in m.kv_cache_spec()["layer_shapes"]] == [True, False, True]
    assert preset("fizunex-8b", num_hidden_layers=4).layer_specs[3].mixer == "parallel"
    assert set(FizunexForCausalLM.native_sources) <= {p.stem for p in b.CSRC.glob("*.cu")}


@pytest.mark.timeout(120)
def test_server_from_its_command_line(tmp_path):
    import argparse
    import asyncio
    httpx = pytest.importorskip("httpx")
    from vllm_gcu_b200.entrypoints.api_server import (ByteTokenizer, add_engine_arguments,
                                                      build_app, make_engine)
    cfg, w, path = build(tmp_path, "prime", seed=12)
    ap = argparse.ArgumentParser()
    add_engine_arguments(ap)
    eng, mc = make_engine(ap.parse_args(["--model", path, "--device", "cpu", "--dtype", "float32",
                                         "--max-num-seqs", "4", "--max-model-len", "128"]))
    app = build_app(eng, ByteTokenizer(mc.vocab_size), "fizunex")
    prompts = [tokens_for(cfg, n, n) for n in (5, 33)]

    async def call():
        async with httpx.AsyncClient(transport=httpx.ASGITransport(app=app),
                                     base_url="http://t") as c:
            return (await c.post("/v1/completions", json={
                "prompt": prompts, "max_tokens": 6, "temperature": 0.0, "ignore_eos": True})).json()
    try:
        out = asyncio.run(call())
    finally:
        eng.shutdown()
    assert [c["token_ids"] for c in out["choices"]] == [greedy(cfg, w, p, 6) for p in prompts]
