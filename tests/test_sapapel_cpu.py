"""Sapapel on the CPU path: every mechanism against the oracle's equations, then the engine's step
(cache, block state, batches, portions) and its generation path against whole-sequence evaluation."""
import dataclasses
import json
import math

import pytest
import torch

import sapapel_oracle as O
from sapapel_cases import (CONFIGS, errors, layer, mixed_steps, model_config, oracle,
                           peaked_weights, portions, replayer, run, spread, tokens_for,
                           write_checkpoint)

TOL = 2e-5


def _checkpoint(tmp_path, name, seed=0, sharp=None):
    cfg = CONFIGS[name]
    w = O.random_model(cfg, seed) if sharp is None else peaked_weights(cfg, seed, sharp)
    return cfg, w, write_checkpoint(tmp_path / name, cfg, w)


# -- mechanisms -------------------------------------------------------------------------
def test_token_shift_rows_and_block_state():
    from vllm_gcu_b200.ops import ref
    g = torch.Generator().manual_seed(0)
    H, bs = 12, 4
    mu = torch.rand(H, generator=g)
    a, b = torch.randn(11, H, generator=g), torch.randn(6, H, generator=g)
    want = {0: O.token_shift(a, mu), 1: O.token_shift(b, mu)}
    bt = torch.tensor([[5, 2, 7], [1, 6, 0]], dtype=torch.int32)
    state = torch.full((8, H), 99.0)                 # what an earlier owner left behind
    cache = torch.zeros(8, bs, 4)
    kv, nw = torch.randn(11, 4, generator=g), torch.ones(4)
    at = [0, 0]
    rows = (a, b)
    got = {0: [], 1: []}
    for step in ([(0, 3)], [(1, 1), (0, 2)], [(0, 1), (1, 4)], [(1, 1), (0, 1)], [(0, 4)]):
        step = sorted(step, key=lambda s: s[1] != 1)           # single tokens first
        nd = sum(1 for s in step if s[1] == 1)
        x = torch.cat([rows[r][at[r]:at[r] + n] for r, n in step])
        pos = torch.cat([torch.arange(at[r], at[r] + n) for r, n in step])
        slots = torch.cat([bt[r][torch.arange(at[r], at[r] + n) // bs].long() * bs
                           + torch.arange(at[r], at[r] + n) % bs for r, n in step])
        cu = torch.tensor([0] + [n for _, n in step[nd:]]).cumsum(0).int() if step[nd:] else None
        tables = torch.stack([bt[r] for r, _ in step])
        h = ref.token_shift(x, mu, torch.float32, state, tables, pos, nd, cu, bs)
        ref.latent_cache(kv[:x.shape[0]], nw, 1e-5, cache, slots, x, state, nd, cu)
        k = 0
        for r, n in step:
            got[r].append(h[k:k + n])
            k += n
            at[r] += n
    for r in (0, 1):
        assert torch.allclose(torch.cat(got[r]), want[r], atol=1e-6)
    # a full block keeps its last row
    assert torch.equal(state[5], a[3]) and torch.equal(state[2], a[7])


@pytest.mark.parametrize("routed", [False, True])
def test_post_norm_depth_average_and_final_norm(routed):
    from vllm_gcu_b200.ops import ref
    g = torch.Generator().manual_seed(1)
    T, H, n, k = 5, 10, 3, 2
    x, hist = torch.randn(T, H, generator=g), torch.randn(4, T, H, generator=g)
    gain, fgain = torch.tensor(1.3), torch.tensor(0.7)
    w = torch.randn(n + 1, generator=g)
    if routed:
        ys, pos = torch.randn(T * k + 3, H + 2, generator=g), torch.randperm(T * k + 3)[:T * k]
        y = ys[pos].view(T, k, -1).sum(1)[:, :H]
        kw = dict(pos_of=pos.int(), k=k)
    else:
        ys = y = torch.randn(T, H, generator=g)
        kw = {}
    r = O.post_norm(x, y, gain, 2.5, 1e-3)
    avg = O.depth_average([*hist[:n], r], w)
    out, res, lo = torch.empty(T, H), torch.empty(T, H), torch.empty(T, H)
    ref.post_norm(x, ys, gain, 2.5, 1e-3, res=res, hist=hist, n=n, weights=w, avg=out,
                  final_gain=fgain, lo=lo, **kw)
    assert torch.allclose(res, r, atol=1e-5) and torch.allclose(out, avg, atol=1e-5)
    assert torch.allclose(lo, O.scalar_norm(avg, fgain, 1e-3), atol=1e-5)
    ref.post_norm(x, ys, gain, 2.5, 1e-3, lo=lo, **kw)
    assert torch.allclose(lo, r, atol=1e-5)


@pytest.mark.parametrize("top", [1, 3, 7])
def test_router_and_input_weighted_experts(top):
    from vllm_gcu_b200.layers.moe import InputWeightedMoE, select_experts
    from vllm_gcu_b200.config import ModelConfig
    g = torch.Generator().manual_seed(2)
    T, H, E, F = 9, 24, 7, 20
    w = {"router": torch.randn(E, H, generator=g)}
    moe = InputWeightedMoE(E, H, F, torch.float32, "cpu")
    for e in range(E):
        for n, s in (("gate", (F, H)), ("up", (F, H)), ("down", (H, F))):
            w[f"e{e}.{n}"] = torch.randn(*s, generator=g) * 0.3
            assert moe.load_expert_weight(e, n, w[f"e{e}.{n}"])
    x = torch.randn(T, H, generator=g)
    rc = ModelConfig(num_experts=E, num_experts_per_tok=top, scoring_func="sigmoid",
                     norm_topk_prob=False)
    s, ids = select_experts(x @ w["router"].T, rc)
    ws, wi = O.route(x, w["router"], top)
    assert torch.equal(ids.long().sort(-1).values, wi.sort(-1).values)
    assert torch.allclose(s.sort(-1).values, ws.sort(-1).values, atol=1e-6)
    y, pos = moe(x, s, ids)
    got = y[pos.long()].view(T, top, H).sum(1)
    want = O.moe(x, w, top)
    assert torch.allclose(got, want, atol=1e-4)
    # weighting the output instead is something else
    plain = O.moe(x, {**w, "router": w["router"] * 1e3}, top)
    assert not torch.allclose(plain, want, atol=1e-2)


def test_latent_attention_layer_matches_expanded_heads():
    """One portion through the layer: absorbed products over the padded cache rows against keys and
    values expanded per head."""
    from vllm_gcu_b200.config import LayerSpec
    from vllm_gcu_b200.layers.attention import AttentionMetadata
    from vllm_gcu_b200.layers.latent import LatentAttention
    g = torch.Generator().manual_seed(3)
    H, T, bs = 20, 13, 4
    for heads, dim, vdim, rank, scale in ((3, 6, 10, 18, 0.7), (1, 4, 4, 4, 1.0)):
        m = LatentAttention(LayerSpec("latent_attention", heads, dim, vdim, rank, scale), H, 1e-3,
                            torch.float32, "cpu", "x")
        w = {"q": (heads * dim, H), "dkv": (rank, H), "uk": (heads * dim, rank),
             "uv": (heads * vdim, rank), "g": (heads * vdim, H), "o": (H, heads * vdim)}
        w = {k: torch.randn(*s, generator=g) * s[1] ** -0.5 for k, s in w.items()}
        w["dkv.norm"] = 1.0 + torch.rand(rank, generator=g)
        for k, v in w.items():
            m.load_weight(k, v)
        m.finalize()
        h = torch.randn(T, H, generator=g)
        cache = torch.full((6, bs, m.W), 7.0)
        bt = torch.tensor([[4, 1, 3, 0]], dtype=torch.int32)
        pos = torch.arange(T)
        md = AttentionMetadata(
            num_tokens=T, num_decodes=0, num_prefills=1, num_decode_tokens=0, positions=pos,
            slot_mapping=bt[0][pos // bs].long() * bs + pos % bs, block_tables=bt,
            seq_lens=torch.tensor([T], dtype=torch.int32),
            cu_q_prefill=torch.tensor([0, T], dtype=torch.int32), q_lens_cpu=[T],
            seq_lens_cpu=[T], max_seq_len=T)
        got = m(h, cache, md)
        assert torch.allclose(got, O.latent_attention(h, w, heads, dim, vdim, scale, 1e-3),
                              atol=1e-4)


# -- configuration and weights ----------------------------------------------------------
def test_configuration_reader():
    from vllm_gcu_b200.config import ModelConfig, preset
    c = ModelConfig.from_hf_dict(CONFIGS["uneven"], dtype="float32")
    assert c.architecture == "SapapelForCausalLM" and c.num_hidden_layers == 3
    assert (c.vocab_size, c.hidden_size, c.rms_norm_eps, c.residual_alpha) == (151, 72, 1e-4, 1.7)
    s = c.layer_specs
    assert [x.has_mlp for x in s] == [True, False, True]
    assert (s[1].num_heads, s[1].head_dim, s[1].v_head_dim, s[1].kv_lora_rank, s[1].scale) == \
        (5, 16, 8, 40, 0.2)
    assert (s[2].num_experts, s[2].num_experts_per_tok, s[2].moe_intermediate_size) == (3, 3, 40)
    assert c.kv_bytes_per_token() == (36 + 40 + 24) * 4
    for bad in ({"type": "convolution"}, {"mlp": {"kind": "dense"}},
                {"mlp": {"kind": "moe", "router": {"experts": 2, "top": 3}, "expert": {"ff": 4}}}):
        d = json.loads(json.dumps(CONFIGS["ones"]))
        d["layers"][0].update(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(d)
    p = preset("tiny-sapapel", num_hidden_layers=5, dtype="float32")
    assert p.num_hidden_layers == 5 == len(p.layer_specs)


def test_missing_and_extra_tensors(tmp_path):
    from vllm_gcu_b200.config import ModelConfig
    from vllm_gcu_b200.models import build_model
    cfg = CONFIGS["uneven"]
    w = O.random_model(cfg)
    m = build_model(ModelConfig.from_hf_dict(cfg, dtype="float32"), "cpu")
    assert "l9.shift" not in m.load_weights({**w, "l9.shift": torch.zeros(3)}.items())
    w.pop("l2.mlp.e1.up")
    with pytest.raises(ValueError, match="l2.mlp.e1.up"):
        build_model(ModelConfig.from_hf_dict(cfg, dtype="float32"), "cpu").load_weights(w.items())


def test_unsupported_combinations_are_refused():
    from vllm_gcu_b200.engine.llm import LLM
    with pytest.raises(ValueError, match="draft"):
        LLM("tiny-sapapel", device="cpu", dtype="float32", speculative_method="ngram",
            num_speculative_tokens=2, max_num_seqs=2, max_model_len=64)
    with pytest.raises(ValueError, match="bfloat16 or float32"):
        LLM("tiny-sapapel", device="cpu", dtype="float16", max_num_seqs=2, max_model_len=64)


# -- the engine's step ------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_portions_and_decoding_match_the_oracle(tmp_path, name):
    cfg, w, path = _checkpoint(tmp_path, name)
    toks = tokens_for(cfg, 53)
    want = oracle(cfg, w, {"a": toks})["a"]
    rp = replayer(path, "cpu", max_tokens=128)
    for sizes in ([53], [1], [2], [3, 2, 7], [16, 1], [31, 2, 1], [17, 15, 16]):
        got = run(rp, {"a": toks}, [[("a", n)] for n in portions(53, sizes)])["a"]
        assert errors(got, want).max() < TOL, sizes


def test_far_keys_at_page_borders(tmp_path):
    """Heads that read one key each: swapping the token at a far position, at the edges of pages
    and at the start changes late logits, and the engine follows the oracle either way, in a
    prompt and in decoding."""
    cfg, w, path = _checkpoint(tmp_path, "uneven", seed=4, sharp=6.0)
    n = 150
    base = tokens_for(cfg, n, 7)
    rp = replayer(path, "cpu", max_tokens=256)
    ref_logits = O.forward(cfg, w, base)
    moved = 0
    for p in (0, 1, 15, 16, 17, 31, 32, 63, 64, 127):
        toks = list(base)
        toks[p] = (toks[p] + 1) % cfg["vocab"]
        want = O.forward(cfg, w, toks)
        moved += int((errors(want, ref_logits)[-30:] > 1e-2).any())
        for sizes in ([n], [n - 6, 1, 1, 1, 1, 1, 1]):
            got = run(rp, {"a": toks}, [[("a", c)] for c in portions(n, sizes)])["a"]
            assert errors(got, want).max() < 1e-3, (p, sizes)
    assert moved >= 8          # the test would notice a lost key


def test_batches_match_each_request_alone_and_blocks_are_used_again(tmp_path):
    cfg, w, path = _checkpoint(tmp_path, "uneven", seed=5)
    prompts = {f"r{i}": tokens_for(cfg, n, i) for i, n in
               enumerate((1, 40, 2, 65, 17, 90, 33, 3, 64, 16))}
    want = oracle(cfg, w, prompts)
    # room for about four requests: later ones get the blocks of earlier ones
    rp = replayer(path, "cpu", max_tokens=320)
    steps = mixed_steps(prompts)
    assert max(len(s) for s in steps) >= 3
    used = set()
    real = rp.engine.scheduler.kv.pool.allocate

    def allocate(k):
        ids = real(k)
        used.update(ids or ())
        return ids
    rp.engine.scheduler.kv.pool.allocate = allocate
    got = run(rp, prompts, steps)
    for k in prompts:
        assert errors(got[k], want[k]).max() < TOL, k
    assert sum(-(-len(p) // 16) for p in prompts.values()) > len(used)
    assert rp.engine.scheduler.kv.pool.num_free_blocks == 20 and not rp.live


def test_a_request_can_pause_while_others_run(tmp_path):
    cfg, w, path = _checkpoint(tmp_path, "odd", seed=6)
    prompts = {"a": tokens_for(cfg, 40, 1), "b": tokens_for(cfg, 47, 2)}
    want = oracle(cfg, w, prompts)
    rp = replayer(path, "cpu", max_tokens=128)
    steps = [[("a", 17)], [("b", 15)], [("b", 2)], [("b", 1)], [("a", 1)], [("b", 14), ("a", 2)],
             [("b", 15)], [("a", 20)]]
    got = run(rp, prompts, steps)
    assert all(errors(got[k], want[k]).max() < TOL for k in prompts)


def test_long_decoding(tmp_path):
    cfg, w, path = _checkpoint(tmp_path, "ones", seed=7)
    prompts = {"a": tokens_for(cfg, 210, 1), "b": tokens_for(cfg, 190, 2)}
    want = oracle(cfg, w, prompts)
    rp = replayer(path, "cpu", max_tokens=512)
    steps = spread([("a", 2)] + [("a", 1)] * 208, [("b", 1)] * 190)
    got = run(rp, prompts, steps)
    assert all(errors(got[k], want[k]).max() < TOL for k in prompts)


def test_a_planted_mistake_shows(tmp_path):
    """The comparison is sharp enough: oracles with one mistake each are told apart from the
    engine."""
    cfg, w, path = _checkpoint(tmp_path, "uneven", seed=8)
    toks = tokens_for(cfg, 30)
    got = run(replayer(path, "cpu", max_tokens=64), {"a": toks}, [[("a", 30)]])["a"]
    assert errors(got, O.forward(cfg, w, toks)).max() < TOL
    shift, attend, route = O.token_shift, O.latent_attention, O.route
    try:
        O.token_shift = lambda h, mu: torch.cat([h[:1], shift(h, mu)[1:]])
        assert errors(got, O.forward(cfg, w, toks))[0] > 100 * TOL
        O.token_shift = shift
        O.latent_attention = lambda h, *a: torch.cat([attend(h, *a)[:-1], attend(h[1:], *a)[-1:]])
        assert errors(got, O.forward(cfg, w, toks))[-1] > 100 * TOL
        O.latent_attention = attend
        O.route = lambda *a: (lambda s, i: (s / s.sum(-1, keepdim=True), i))(*route(*a))
        assert errors(got, O.forward(cfg, w, toks)).min() > 100 * TOL
    finally:
        O.token_shift, O.latent_attention, O.route = shift, attend, route


def test_replayer_rejects_bad_steps(tmp_path):
    cfg, w, path = _checkpoint(tmp_path, "ones")
    rp = replayer(path, "cpu", max_tokens=64)
    with pytest.raises(ValueError, match="vocabulary"):
        rp.step([{"id": "a", "tokens": [cfg["vocab"]]}])
    with pytest.raises(ValueError, match="wanted"):
        rp.step([{"id": "b", "tokens": [1], "want": [1]}])
    with pytest.raises(ValueError, match="longer"):
        rp.step([{"id": "c", "tokens": [1] * 65}])


# -- generation -------------------------------------------------------------------------
def greedy(cfg, w, prompt, n):
    toks, out = list(prompt), []
    for _ in range(n):
        out.append(int(O.forward(cfg, w, toks)[-1].argmax()))
        toks.append(out[-1])
    return out


@pytest.mark.parametrize("kw", [
    dict(), dict(async_scheduling=True), dict(max_num_batched_tokens=16, max_num_seqs=3),
    dict(num_gpu_blocks=7), dict(num_gpu_blocks=7, num_cpu_blocks=32),
    dict(num_scheduler_steps=3)],
    ids=["plain", "async", "chunked", "preempt", "swap", "multistep"])
def test_greedy_generation_through_the_engine(tmp_path, kw):
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    cfg, w, path = _checkpoint(tmp_path, "uneven", seed=9)
    prompts = [tokens_for(cfg, n, 20 + n) for n in (1, 18, 37, 16, 50)]
    llm = LLM(path, device="cpu", dtype="float32", **{
        **dict(max_num_seqs=4, max_model_len=128, num_gpu_blocks=64), **kw})
    outs = llm.generate(prompts, SamplingParams(max_tokens=14, temperature=0.0, ignore_eos=True))
    assert [o.outputs[0].token_ids for o in outs] == [greedy(cfg, w, p, 14) for p in prompts]
    sch = llm.engine.scheduler
    if kw.get("num_gpu_blocks") == 7:
        assert sch.num_preemptions > 0
        assert (sch.num_swaps > 0) == ("num_cpu_blocks" in kw)


def test_prefix_cache_hits_bring_the_state_along(tmp_path):
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    cfg, w, path = _checkpoint(tmp_path, "odd", seed=10)
    llm = LLM(path, device="cpu", dtype="float32", max_num_seqs=4, max_model_len=128,
              num_gpu_blocks=64)
    sp = SamplingParams(max_tokens=5, temperature=0.0, ignore_eos=True)
    head = tokens_for(cfg, 48, 1)
    for tail in ([3], [5, 9], tokens_for(cfg, 20, 2)):
        o = llm.generate([head + tail], sp)[0]
        assert o.outputs[0].token_ids == greedy(cfg, w, head + tail, 5)
    assert o.num_cached_tokens == 48


def test_sampling_and_logprobs(tmp_path):
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    cfg, w, path = _checkpoint(tmp_path, "ones", seed=11)
    llm = LLM(path, device="cpu", dtype="float32", max_num_seqs=4, max_model_len=64)
    p = tokens_for(cfg, 9)
    a = llm.generate([p], SamplingParams(max_tokens=6, temperature=0.8, seed=3, ignore_eos=True))
    b = llm.generate([p], SamplingParams(max_tokens=6, temperature=0.8, seed=3, ignore_eos=True))
    assert a[0].outputs[0].token_ids == b[0].outputs[0].token_ids
    o = llm.generate([p], SamplingParams(max_tokens=1, temperature=0.0, logprobs=2,
                                         prompt_logprobs=0, ignore_eos=True))[0]
    lp = torch.log_softmax(O.forward(cfg, w, p), -1)
    t = o.outputs[0].token_ids[0]
    assert math.isclose(o.outputs[0].logprobs[0][t], float(lp[-1, t]), abs_tol=1e-4)
    for i in range(1, 9):
        assert math.isclose(o.prompt_logprobs[i][p[i]], float(lp[i - 1, p[i]]), abs_tol=1e-4)


def test_partial_library_name_and_sources_exist():
    from vllm_gcu_b200.csrc import build
    from vllm_gcu_b200.models.sapapel import SapapelForCausalLM
    have = {p.stem for p in build.CSRC.glob("*.cu")}
    assert set(SapapelForCausalLM.native_sources) <= have
    assert build.partial_lib_path(["a", "b"]) == build.partial_lib_path(["b", "a"])
    assert build.partial_lib_path(["a"]) != build.LIB_PATH


def test_layer_spec_is_frozen():
    from vllm_gcu_b200.config import LayerSpec
    with pytest.raises(dataclasses.FrozenInstanceError):
        LayerSpec("latent_attention", 1, 1, 1, 1, 1.0).scale = 2.0
    assert not LayerSpec("latent_attention", 1, 1, 1, 1, 1.0).has_mlp
    assert layer(1, 1, 1, 1, 1.0)["mlp"] is None
    assert model_config(8, 4, 1.0, 1e-5, [])["layers"] == []


@pytest.mark.timeout(120)
def test_server_from_its_command_line(tmp_path):
    import argparse
    import asyncio
    httpx = pytest.importorskip("httpx")
    from vllm_gcu_b200.entrypoints.api_server import (ByteTokenizer, add_engine_arguments,
                                                      build_app, make_engine)
    cfg, w, path = _checkpoint(tmp_path, "prime", seed=12)
    ap = argparse.ArgumentParser()
    add_engine_arguments(ap)
    eng, mc = make_engine(ap.parse_args(["--model", path, "--device", "cpu", "--dtype", "float32",
                                         "--max-num-seqs", "4", "--max-model-len", "128"]))
    app = build_app(eng, ByteTokenizer(mc.vocab_size), "sapapel")
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
