"""Fepopel on the CPU path: every mechanism against the oracle's equations, then the engine's step
(caches per layer run, batches, portions) and its generation path against whole-sequence
evaluation."""
import json
import math

import pytest
import torch

import fepopel_oracle as O
from fepopel_cases import (CONFIGS, build, chunk_edges, chunked, dense, errors, greedy, latent,
                           mixed_steps, model_config, moe, oracle, paged_batch, peaked_model,
                           portions, replayer, run, spread, tokens_for, write_checkpoint)

TOL = 3e-5


def gen(seed):
    return torch.Generator().manual_seed(seed)


def one_request(T, bs, blocks):
    """Metadata of one portion of T tokens from position 0 in the given blocks."""
    from vllm_gcu_b200.layers.attention import AttentionMetadata
    bt = torch.tensor([blocks], dtype=torch.int32)
    pos = torch.arange(T)
    return AttentionMetadata(
        num_tokens=T, num_decodes=0, num_prefills=1, num_decode_tokens=0, positions=pos,
        slot_mapping=bt[0][pos // bs].long() * bs + pos % bs, block_tables=bt,
        seq_lens=torch.tensor([T], dtype=torch.int32),
        cu_q_prefill=torch.tensor([0, T], dtype=torch.int32), q_lens_cpu=[T], seq_lens_cpu=[T],
        max_seq_len=T)


# -- mechanisms -------------------------------------------------------------------------
@pytest.mark.parametrize("heads,dim,rot,vdim,rank,scale", [(3, 6, 4, 10, 18, 0.7),
                                                           (1, 4, 2, 4, 4, 1.0),
                                                           (2, 5, 8, 3, 7, 0.4)])
def test_latent_attention_matches_expanded_heads(heads, dim, rot, vdim, rank, scale):
    from vllm_gcu_b200.config import LayerSpec
    from vllm_gcu_b200.layers.basic import build_cos_sin_cache
    from vllm_gcu_b200.layers.latent import LatentAttention
    g = gen(3)
    H, T, bs, base = 20, 13, 4, 50.0
    spec = LayerSpec("latent_attention", heads, dim, vdim, rank, scale, rot_dim=rot, sink=True,
                     head_gate=True)
    m = LatentAttention(spec, H, 1e-3, torch.float32, "cpu", "x",
                        build_cos_sin_cache(rot, 64, base, dtype=torch.float64).float())
    w = {"q": (heads * (dim + rot), H), "dkv": (rank + rot, H), "uk": (heads * dim, rank),
         "uv": (heads * vdim, rank), "g": (heads, H), "o": (H, heads * vdim)}
    w = {k: torch.randn(*s, generator=g) * s[1] ** -0.5 for k, s in w.items()}
    w["q"] *= 3.0
    w["dkv.norm"] = 1.0 + torch.rand(rank, generator=g)
    w["sink"] = torch.linspace(-3.0, 3.0, heads)
    assert m.tensor_names() == set(w)
    for k, v in w.items():
        assert m.load(k, v)
    m.finalize()
    h = torch.randn(T, H, generator=g)
    got = m(h, torch.full((6, bs, m.W), 7.0), one_request(T, bs, [4, 1, 3, 0]))
    args = (heads, dim, rot, vdim, rank, scale, base, 1e-3)
    want = O.latent_attention(h, w, *args)
    assert torch.allclose(got, want, atol=1e-4)
    # what a lost sink, a lost gate and another base would give is something else
    for other in ({**w, "sink": w["sink"] * 0 - 90.0}, {**w, "g": w["g"] * 0}):
        assert not torch.allclose(O.latent_attention(h, other, *args), want, atol=1e-2)
    if rot > 2:         # the first pair's angle is the position whatever the base
        assert not torch.allclose(O.latent_attention(h, w, *args[:6], 5.0, 1e-3), want, atol=1e-3)


@pytest.mark.parametrize("heads,kv,dim,vdim,size", [(4, 2, 6, 10, 5), (3, 3, 8, 4, 1), (6, 1, 5, 5, 7),
                                                    (2, 1, 4, 6, 64)])
def test_chunk_attention_matches_its_equations(heads, kv, dim, vdim, size):
    from vllm_gcu_b200.config import AttentionSpec
    from vllm_gcu_b200.layers.key_attention import ChunkAttention
    from vllm_gcu_b200.layers.mixer import MixerBlock
    g = gen(4)
    H, T, bs, cap = 20, 23, 4, 3.0
    part = ChunkAttention(AttentionSpec(heads, kv, dim, 0.8, v_head_dim=vdim, softcap=cap,
                                        chunk=size), 1e-3, torch.float32, "cpu", "x")
    m = MixerBlock([("", 1.0, part)], H, torch.float32, "cpu", "x")
    w = {"q": (heads * dim, H), "k": (kv * dim, H), "v": (kv * vdim, H), "o": (H, heads * vdim)}
    w = {k: torch.randn(*s, generator=g) * s[1] ** -0.5 for k, s in w.items()}
    w.update({"q.norm": 2.0 + torch.rand(dim, generator=g), "k.norm": torch.rand(dim, generator=g)})
    assert m.tensor_names() == set(w)
    for k, v in w.items():
        assert m.load(k, v)
    h = torch.randn(T, H, generator=g)
    cache = torch.full((2, 8, bs, *part.cache_shape()), 7.0)
    got = m(h, one_request(T, bs, [4, 1, 3, 0, 6, 7]), cache, None)
    args = (heads, kv, dim, vdim, 0.8)
    assert torch.allclose(got, O.chunk_attention(h, w, *args, cap, size, 1e-3), atol=1e-4)
    if size < T:
        assert not torch.allclose(got, O.chunk_attention(h, w, *args, cap, size + 1, 1e-3),
                                  atol=1e-2)
    if size > 1:
        assert not torch.allclose(got, O.chunk_attention(h, w, *args, 1e6, size, 1e-3), atol=1e-2)


@pytest.mark.parametrize("chunk", [0, 24, 16, 40, 129])
def test_keys_at_chunk_edges(chunk):
    """Keys that stand out just inside and just outside a chunk, for portions and single tokens."""
    from vllm_gcu_b200.ops import ref
    ql, sl = [1, 1, 1, 70, 2], [49, 48, 130, 131, 41]
    q, kc, vc, bt, s, cu = paged_batch(4, 2, 12, ql, sl, chunk, torch.float32, seed=chunk)
    got = ref.any_attention(q, kc, vc, bt, s, 3, cu[3:] - cu[3], 0.5, softcap=6.0, chunk=chunk,
                            out_dim=10)
    for b, n in enumerate(sl):
        at = torch.arange(n)
        k, v = (c[bt[b, at // 16].long(), at % 16].double() for c in (kc, vc))
        for i in range(ql[b]):
            pos = n - ql[b] + i
            for a in range(4):
                sc = 6.0 * torch.tanh(0.5 * (k[:, a // 2] @ q[int(cu[b]) + i, a].double()) / 6.0)
                ok = (at <= pos) & (at // chunk == pos // chunk if chunk else at >= 0)
                want = O.softmax_values(sc.masked_fill(~ok, -math.inf)[None], v[:, a // 2])[0]
                assert torch.allclose(got[int(cu[b]) + i, a].double(), want[:10], atol=1e-4)


@pytest.mark.parametrize("top,shared,scale", [(1, 0, 1.0), (3, 12, 2.5), (7, 5, 0.3)])
def test_router_experts_and_shared_expert(top, shared, scale):
    from vllm_gcu_b200.layers.moe import GatedSharedMoE
    from vllm_gcu_b200.ops import ref
    g = gen(2)
    T, H, E, F = 9, 24, 7, 20
    m = GatedSharedMoE(E, top, scale, H, F, shared, torch.float32, "cpu", "x")
    shapes = {"router": (E, H), **{f"e{e}.up": (F, H) for e in range(E)},
              **{f"e{e}.down": (H, F) for e in range(E)}}
    if shared:
        shapes.update({"shared.up": (shared, H), "shared.down": (H, shared), "shared.sg": (1, H)})
    w = {k: torch.randn(*s, generator=g) * s[1] ** -0.5 for k, s in shapes.items()}
    assert m.tensor_names() == set(w)
    assert all(m.load(k, v) for k, v in w.items())
    assert not m.load("e0.gate", w["e0.up"]) and not m.load(f"e{E}.up", w["e0.up"])
    h = torch.randn(T, H, generator=g)
    y, rows = m(h)
    # as the residual kernel takes it: the row before its norm, read back through the norm
    x, lo, one = torch.zeros(T, H), torch.empty(T, H), torch.ones(H)
    ref.add_normed(x, y, one, None, 1e-6, lo, layer_norm=False, **rows)
    want = O.moe(h, w, top, scale)
    assert torch.allclose(lo, O.rms(want, one, 1e-6), atol=1e-4)
    if shared:
        plain = O.moe(h, {**w, "shared.sg": w["shared.sg"] * 0}, top, scale)
        assert not torch.allclose(plain, want, atol=1e-2)


def test_residual_rows_and_norms():
    from vllm_gcu_b200.ops import ref
    g = gen(1)
    T, H = 5, 10
    e, y, x = (torch.randn(T, H, generator=g) for _ in range(3))
    step, w, wb = (torch.randn(H, generator=g) for _ in range(3))
    a, lo = ref.start_rows(e, 2.5, step, w, 1e-3)
    assert torch.allclose(a, e * 2.5 + step) and torch.allclose(lo, O.rms(a, w, 1e-3), atol=1e-5)
    a, lo = ref.start_rows(e, 2.5)
    assert torch.allclose(a, e * 2.5) and torch.equal(a, lo)
    out = torch.empty(T, H)
    ref.add_normed(x, y, wb, None, 1e-3, lo, out=out, layer_norm=False, final_weight=w, step=step)
    want = x + O.rms(y, wb, 1e-3) + step
    assert torch.allclose(out, want, atol=1e-5)
    assert torch.allclose(lo, O.rms(want, w, 1e-3), atol=1e-5)


def test_rotary_table_is_exact_far_out():
    from vllm_gcu_b200.layers.basic import build_cos_sin_cache
    t = build_cos_sin_cache(12, 100001, 1e4, dtype=torch.float64).float()
    for p in (0, 1, 4097, 100000):
        for i in range(6):
            a = p * 1e4 ** (-2.0 * i / 12)
            assert math.isclose(t[p, i], math.cos(a), abs_tol=1e-6)
            assert math.isclose(t[p, 6 + i], math.sin(a), abs_tol=1e-6)


# -- configuration and weights ----------------------------------------------------------
def test_configuration_reads_every_number():
    from vllm_gcu_b200.config import AttentionSpec, ModelConfig, preset
    c = ModelConfig.from_hf_dict(CONFIGS["uneven"], dtype="float32")
    assert c.architecture == "FepopelForCausalLM" and c.num_hidden_layers == 4
    assert (c.vocab_size, c.hidden_size, c.rms_norm_eps, c.embed_scale) == (151, 72, 1e-4, 3.0)
    assert c.layer_specs[0].parts == (("", 1.0, AttentionSpec(
        6, 3, 20, 0.3, v_head_dim=28, softcap=4.0, chunk=24)),)
    s = c.layer_specs[1]
    assert (s.num_heads, s.head_dim, s.rot_dim, s.v_head_dim, s.kv_lora_rank, s.scale, s.rot_base,
            s.sink, s.head_gate) == (3, 12, 6, 20, 36, 0.31, 500.0, True, True)
    assert (s.num_experts, s.num_experts_per_tok, s.moe_intermediate_size,
            s.shared_intermediate_size, s.router_scale) == (5, 2, 24, 20, 1.7)
    assert [x.has_mlp for x in c.layer_specs] == [True, True, False, True]
    assert c.loop == (1, 3, 3)
    assert c.layer_runs == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None),
                            (3, None)]
    # a token's cache: every run of a layer counts
    assert c.kv_bytes_per_token() == 4 * (3 * (20 + 28) + 3 * (36 + 6 + 40 + 10) + 24 + 4)
    plain = ModelConfig.from_hf_dict(CONFIGS["prime"])
    assert plain.loop is None and plain.layer_runs == [(0, None), (1, None), (2, None)]
    short = preset("tiny-fepopel", num_hidden_layers=2, dtype="float32")
    assert short.loop == (1, 2, 2) and len(short.layer_runs) == 3
    assert preset("tiny-fepopel", num_hidden_layers=1, dtype="float32").loop is None
    for change, msg in (({"type": "convolution"}, "unknown mixer"),
                        ({"mlp": {"kind": "sparse"}}, "unknown feed-forward"),
                        ({"mlp": moe(2, 3, 4)}, "experts per token")):
        d = json.loads(json.dumps(CONFIGS["ones"]))
        d["layers"][0].update(change)
        with pytest.raises(ValueError, match=msg):
            ModelConfig.from_hf_dict(d)
    d = json.loads(json.dumps(CONFIGS["ones"]))
    d["layers"][0]["mixer"]["rot"]["dims"] = 4
    with pytest.raises(ValueError, match="rotated"):
        ModelConfig.from_hf_dict(d)
    for loop in ((0, 3, 2), (1, 1, 2), (0, 2, 0)):
        with pytest.raises(ValueError, match="loop"):
            ModelConfig.from_hf_dict({**CONFIGS["ones"],
                                      "loop": dict(zip(("start", "stop", "times"), loop))})


def test_missing_extra_and_misshapen_tensors():
    from vllm_gcu_b200.config import ModelConfig
    from vllm_gcu_b200.models import build_model
    cfg = CONFIGS["uneven"]
    w = O.random_model(cfg)
    m = build_model(ModelConfig.from_hf_dict(cfg, dtype="float32"), "cpu")
    extra = {k: torch.zeros(3) for k in ("l9.norm1", "l2.norm2", "l3.mlp.shared.up", "l0.mix.sink",
                                         "l0.mlp.e0.up", "l1.mlp.e5.up", "other")}
    assert not set(extra) & m.load_weights({**w, **extra}.items())
    for name in ("l1.mlp.e1.up", "loop.step", "l1.mlp.shared.sg", "l0.mix.q.norm", "l2.mix.sink"):
        with pytest.raises(ValueError, match=name):
            build_model(ModelConfig.from_hf_dict(cfg, dtype="float32"), "cpu").load_weights(
                {k: v for k, v in w.items() if k != name}.items())


def test_unsupported_combinations_are_refused():
    from vllm_gcu_b200.config import ModelConfig
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.models import build_model
    with pytest.raises(ValueError, match="bfloat16 or float32"):
        LLM("tiny-fepopel", device="cpu", dtype="float16", max_num_seqs=2, max_model_len=64)
    llm = LLM("tiny-fepopel", device="cpu", dtype="float32", max_num_seqs=2, max_model_len=64)
    with pytest.raises(ValueError, match="does not ship"):
        llm.engine.attach_kv_connector(object())
    for layer, msg in ((latent(2, 4, 3, 4, 8, 10.0, 1.0), "pair up"),
                       (chunked(3, 2, 4, 4, 8, 1.0, 1.0), "key heads"),
                       (chunked(2, 1, 600, 4, 8, 1.0, 1.0), "at most")):
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


def test_far_keys_page_borders_and_chunk_edges(tmp_path):
    """Heads that read few keys: swapping one token at a far position, at the edges of pages and
    chunks and at the start changes late logits, and the engine follows the oracle either way, in a
    prompt and in decoding."""
    cfg, w, path = build(tmp_path, "uneven", seed=4, weights=peaked_model)
    n = 124                                 # the last chunk of 24 starts at 120
    base = tokens_for(cfg, n, 7)
    rp = replayer(path, "cpu", max_tokens=256)
    before = O.forward(cfg, w, base)
    moved = 0
    at = (0, 1, 15, 16, 17, 31, 64, 95, 96, 119, 120, 121)
    for p in at:
        toks = list(base)
        toks[p] = (toks[p] + 1) % cfg["vocab"]
        want = O.forward(cfg, w, toks)
        moved += int((errors(want, before)[-4:] > 3e-3).any())
        for sizes in ([n], [n - 6, 1, 1, 1, 1, 1, 1]):
            got = run(rp, {"a": toks}, [[("a", c)] for c in portions(n, sizes)])["a"]
            assert errors(got, want).max() < 1e-3, (p, sizes)
    assert moved >= len(at) - 2             # the test would notice a lost key


def test_chunks_hide_what_lies_in_front_of_them(tmp_path):
    """A model of chunked layers alone: a token changes the logits of its chunk and no others."""
    cfg = model_config(60, 24, [chunked(4, 2, 8, 8, 10, 0.5, 5.0, dense(16))] * 2, (0, 1, 2))
    w = O.random_model(cfg, 3)
    path = write_checkpoint(tmp_path / "c", cfg, w)
    rp = replayer(path, "cpu", max_tokens=64)
    a, b = tokens_for(cfg, 34, 1), tokens_for(cfg, 34, 1)
    b[19] = (b[19] + 1) % 60
    got = [run(rp, {"a": t}, [[("a", c)] for c in portions(34, sizes)])["a"]
           for t in (a, b) for sizes in ([34], [7, 2, 1])]
    for x, y in ((got[0], got[2]), (got[1], got[3])):
        same = (x - y).abs().amax(-1) < 1e-5
        assert same[:19].all() and not same[19] and same[20:].all()
    b[10] = (b[10] + 1) % 60
    c = run(rp, {"a": b}, [[("a", 34)]])["a"]
    same = (c - got[2]).abs().amax(-1) < 1e-5
    assert same[:10].all() and not same[10:20].any() and same[20:].all()


def test_batches_match_each_request_alone_and_blocks_are_used_again(tmp_path):
    cfg, w, path = build(tmp_path, "uneven", seed=5)
    prompts = {f"r{i}": tokens_for(cfg, n, i) for i, n in
               enumerate((1, 40, 2, 65, 17, 70, 33, 3, 64, 16))}
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
    prompts = {"a": tokens_for(cfg, 170, 1), "b": tokens_for(cfg, 150, 2)}
    want = oracle(cfg, w, prompts)
    rp = replayer(path, "cpu", max_tokens=512)
    steps = spread([("a", 2)] + [("a", 1)] * 168, [("b", 1)] * 150)
    got = run(rp, prompts, steps)
    assert all(errors(got[k], want[k]).max() < TOL for k in prompts)


def test_every_pass_has_its_own_cache(tmp_path):
    from vllm_gcu_b200.models.fepopel import FepopelForCausalLM
    cfg, w, path = build(tmp_path, "uneven", seed=13)
    rp = replayer(path, "cpu", max_tokens=64)
    model, caches = rp.engine.model, rp.engine.runner.kv_caches
    assert isinstance(model, FepopelForCausalLM) and len(model.layers) == 4
    assert len(caches) == 8 == model.num_local_layers == len({c.data_ptr() for c in caches})
    assert [c.dim() for c in caches] == [5, 3, 3, 3, 3, 3, 3, 3]
    assert model.kv_cache_spec()["layer_shapes"][:3] == [(3, 28), (44,), (52,)]


def test_a_planted_mistake_shows(tmp_path):
    """The comparison is sharp enough: oracles with one mistake each are told apart from the
    engine."""
    cfg, w, path = build(tmp_path, "uneven", seed=8)
    toks = tokens_for(cfg, 30)
    got = run(replayer(path, "cpu", max_tokens=64), {"a": toks}, [[("a", 30)]])["a"]
    assert errors(got, O.forward(cfg, w, toks)).max() < TOL
    real = {n: getattr(O, n) for n in ("rotate", "softmax_values", "same_chunk", "route", "expert",
                                       "layer_runs", "rms", "causal")}
    wrong = {
        "rotate": lambda x, b: torch.cat([real["rotate"](x, b)[:-1], x[-1:]]),
        "softmax_values": lambda s, v, sink=None: real["softmax_values"](s, v),
        "same_chunk": lambda T, n: real["same_chunk"](T + 1, n)[1:, 1:],
        "route": lambda h, r, k, s: real["route"](h, r, k, 1.0),
        "expert": lambda h, up, down: torch.clamp(h @ up.T, min=0.0) @ down.T,
        "layer_runs": lambda c: [(i, 0 if t == 1 else t) for i, t in real["layer_runs"](c)],
        "rms": lambda x, weight, eps: real["rms"](x, weight, 0.0),
        "causal": lambda T: real["causal"](T).tril(-1) | (torch.eye(T) > 0) & (
            torch.arange(T) < T - 1)[:, None],
    }
    for name, f in wrong.items():
        setattr(O, name, f)
        try:
            assert errors(got, O.forward(cfg, w, toks)).max() > 20 * TOL, name
        finally:
            setattr(O, name, real[name])


# -- generation -------------------------------------------------------------------------
@pytest.mark.parametrize("kw", [
    dict(), dict(async_scheduling=True), dict(max_num_batched_tokens=16, max_num_seqs=3),
    dict(num_gpu_blocks=7), dict(num_gpu_blocks=7, num_cpu_blocks=32),
    dict(num_scheduler_steps=3), dict(speculative_method="ngram", num_speculative_tokens=2)],
    ids=["plain", "async", "chunked", "preempt", "swap", "multistep", "draft"])
def test_greedy_generation_through_the_engine(tmp_path, kw):
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    cfg, w, path = build(tmp_path, "uneven", seed=9)
    prompts = [tokens_for(cfg, n, 20 + n) for n in (1, 18, 37, 16, 50)]
    prompts[2][18:36] = prompts[2][:18]                  # repeats itself: draft tokens are proposed
    llm = LLM(path, device="cpu", dtype="float32", **{
        **dict(max_num_seqs=4, max_model_len=128, num_gpu_blocks=64), **kw})
    outs = llm.generate(prompts, SamplingParams(max_tokens=14, temperature=0.0, ignore_eos=True))
    assert [o.outputs[0].token_ids for o in outs] == [greedy(cfg, w, p, 14) for p in prompts]
    sch = llm.engine.scheduler
    if kw.get("num_gpu_blocks") == 7:
        assert sch.num_preemptions > 0
        assert (sch.num_swaps > 0) == ("num_cpu_blocks" in kw)


def test_prefix_cache_hits(tmp_path):
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    cfg, w, path = build(tmp_path, "prime", seed=10)
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


def test_presets_and_native_sources():
    from vllm_gcu_b200.config import preset
    from vllm_gcu_b200.csrc import build as b
    from vllm_gcu_b200.models import build_model
    from vllm_gcu_b200.models.fepopel import FepopelForCausalLM
    m = build_model(preset("tiny-fepopel", dtype="float32"), "cpu")
    m.init_random(0)
    assert [len(s) for s in m.kv_cache_spec()["layer_shapes"]] == [1, 1, 2, 1, 2, 1]
    big = preset("fepopel-16b")
    assert big.num_hidden_layers == 26 and len(big.layer_runs) == 29
    assert big.layer_specs[2].parts[0][2].chunk == 1024
    assert set(FepopelForCausalLM.native_sources) <= {p.stem for p in b.CSRC.glob("*.cu")}
    assert chunk_edges(20, 8) == [0, 1, 7, 8, 9, 15, 16, 17, 19]


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
    app = build_app(eng, ByteTokenizer(mc.vocab_size), "fepopel")
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
