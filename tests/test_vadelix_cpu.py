"""Vadelix on the CPU path: every mechanism against the oracle's equations, then the engine's step
(cache, state slots, batches, portions) and its generation path against whole-sequence evaluation."""
import math

import pytest
import torch

import vadelix_oracle as O
from vadelix_cases import (CONFIGS, Step, biased, build, errors, greedy, mixed_steps,
                           model_config, moe, oracle, peaked_model, portions, replayer, rotary, run,
                           spread, tokens_for, wkv, write_checkpoint)

TOL = 5e-5


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rand(g, *s):
    return torch.randn(*s, generator=g)


# -- mechanisms -------------------------------------------------------------------------
@pytest.mark.parametrize("H,groups", [(12, 1), (12, 4), (15, 5), (7, 7), (7, 1)])
def test_grouped_norm_after_the_sum(H, groups):
    from vllm_gcu_b200.ops import ref
    g, T, k = gen(H), 5, 3
    x, y, w, rows = rand(g, T, H), rand(g, T, H), rand(g, H), rand(g, T * k + 2, H)
    pos = torch.randperm(T * k + 2, generator=g)[:T * k].int()
    row_w, shared = torch.rand(T, k, generator=g), rand(g, T, H)
    out, lo = torch.empty(T, H), torch.empty(T, H)
    ref.add_group_norm(x, None, 0.3, w, groups, 1e-2, lo, out=out)
    assert torch.equal(out, x) and torch.allclose(lo, O.group_norm(x, w, groups, 1e-2), atol=1e-6)
    ref.add_group_norm(x, y, 0.3, w, groups, 1e-2, lo, out=out)
    assert torch.allclose(out, x + 0.3 * y) and torch.allclose(
        lo, O.group_norm(x + 0.3 * y, w, groups, 1e-2), atol=1e-6)
    s = x + 0.3 * ((rows[pos.long()].view(T, k, H) * row_w[..., None]).sum(1) + shared)
    ref.add_group_norm(x, rows, 0.3, w, groups, 1e-2, lo, pos_of=pos, row_w=row_w, shared=shared)
    assert torch.allclose(lo, O.group_norm(s, w, groups, 1e-2), atol=1e-5)
    if 1 < groups < H:      # the grouping matters
        assert (lo - O.group_norm(s, w, 1, 1e-2)).abs().max() > 1e-2


SCHEDULES = [[11], [1] * 11, [2, 3, 1, 5], [8, 2, 1], [1, 1, 9]]


@pytest.mark.parametrize("taps", [1, 2, 3, 5, 8])
@pytest.mark.parametrize("mixes", [0, 3])
def test_input_convolution_portions_and_slots(taps, mixes):
    from vllm_gcu_b200.ops import ref
    g, T, H = gen(taps), 11, 6
    h, w = rand(g, T, H), rand(g, H, taps)
    mu = torch.rand(mixes, H, generator=g) if mixes else None
    c = O.input_conv(h, w)
    want = c if mu is None else torch.stack([c + (O.past(c, 1) - c) * m for m in mu])
    back = taps - (mu is None)
    ring = torch.full((3, back, H), 7.0) if back else None       # what another request has left
    for sizes in SCHEDULES:
        at, got = 0, []
        for n in sizes:
            out = torch.full((T, H) if mu is None else (mixes, T, H), 9.0)[..., :n, :]
            ref.input_conv(h[at:at + n], w.t().contiguous(), mu,
                           Step([(1, at, n)], decodes=int(n == 1 and at % 2 == 0)), ring, out)
            got.append(out)
            at += n
        assert torch.allclose(torch.cat(got, dim=-2), want, atol=1e-5), sizes
    if back:
        assert (ring[0] == 7.0).all() and (ring[2] == 7.0).all()


@pytest.mark.parametrize("yarn", [None, (2.0, 64, 8.0, 0.5), (4.0, 4096, 32.0, 1.0),
                                  (1.0, 100, 1.0, 1.0), (8.0, 7, 3.0, 2.0)])
@pytest.mark.parametrize("dims,base", [(2, 10.0), (12, 500.0), (64, 1e6)])
def test_rotation_table(dims, base, yarn):
    from vllm_gcu_b200.config import AttentionSpec
    from vllm_gcu_b200.layers.key_attention import rotary_table
    table = rotary_table(AttentionSpec(1, 1, dims, 1.0, dims, base, rot_scaling=yarn or ()), 300, "cpu")
    x = rand(gen(dims), 300, 1, dims).double()
    scaling = dict(zip(("factor", "original", "fast", "slow"), yarn)) if yarn else None
    want = O.rotate_halves(x, dims, base, scaling)
    half = dims // 2
    c, s = table[:, None, :half].double(), table[:, None, half:].double()
    u, v = x[..., :half], x[..., half:]
    assert torch.allclose(torch.cat([u * c - v * s, v * c + u * s], -1), want, atol=1e-6)


def test_slopes_and_temperature():
    from vllm_gcu_b200.layers.attention import alibi_slopes
    from vllm_gcu_b200.layers.key_attention import distance_slopes
    for n in (1, 3, 4, 6, 12):
        assert torch.allclose(distance_slopes(n), torch.tensor(O.slopes(n)))
    assert torch.allclose(distance_slopes(8), alibi_slopes(8))
    t = O.temperature(9, 0.5, 4)
    assert torch.allclose(t[:3], torch.ones(3, dtype=torch.float64)) and t[3] == t[6] > t[2]
    assert t[7] > t[6]


def _attention_case(layer, first, H, T, g, sizes, bs=4):
    """Output of the layer's mixer over portions of ``sizes`` through a paged cache, and the
    oracle's; ``first``: (spec, values) of the layer whose values are mixed in."""
    from vllm_gcu_b200.config import ModelConfig
    from vllm_gcu_b200.layers.attention import AttentionMetadata
    from vllm_gcu_b200.layers.key_attention import GroupedAttention, rotary_table
    from vllm_gcu_b200.layers.mixer import MixerBlock
    cfg = ModelConfig.from_hf_dict(model_config(8, H, [layer], 1, 1, 1.0, 1e-3), dtype="float32")
    spec, m = cfg.layer_specs[0].parts[0][2], layer["mixer"]
    part = GroupedAttention(spec, 1e-3, torch.float32, "cpu", "p", rotary_table(spec, 64, "cpu"),
                            first[0] if first else None)
    block = MixerBlock([("", 1.0, part)], H, torch.float32, "cpu", "p")
    shapes = {k[7:]: s for k, s in O.tensor_shapes(model_config(8, H, [layer], 1)).items()
              if k.startswith("l0.mix.")}
    w = {n: (torch.randn(s, generator=g) if s else torch.tensor(0.3))
         * (s[-1] ** -0.5 if len(s) > 1 else 1.0) for n, s in shapes.items()}
    assert block.tensor_names() == set(w) and all(block.load(n, t) for n, t in w.items())
    h = rand(g, T, H)
    wd = {n: t.double() for n, t in w.items()}
    v1 = None if first is None else first[1].double()
    want, _ = O.rotary_attention(h.double(), wd, m, 1e-3, v1) if layer["type"] == "attention" else \
        O.biased_attention(h.double(), wd, m, v1)
    cache = torch.full((2, 10, bs, *part.cache_shape()), 7.0)
    bt = torch.tensor([[4, 1, 3, 0, 6, 8, 2, 9]], dtype=torch.int32)
    got, at = [], 0
    for n in sizes:
        pos = torch.arange(at, at + n)
        slots = bt[0][pos // bs].long() * bs + pos % bs
        values = None
        if first is not None:
            G, V = first[0].num_kv_heads, first[0].v_head_dim
            values = torch.full((10, bs, G, V + 3), 5.0)
            values.view(10 * bs, G, V + 3)[slots, :, :V] = first[1][at:at + n].view(n, G, V)
        md = AttentionMetadata(
            num_tokens=n, num_decodes=int(n == 1), num_prefills=int(n > 1),
            num_decode_tokens=int(n == 1), positions=pos, block_tables=bt, slot_mapping=slots,
            seq_lens=torch.tensor([at + n], dtype=torch.int32),
            cu_q_prefill=torch.tensor([0, n], dtype=torch.int32) if n > 1 else None,
            first_values=values)
        got.append(block(h[at:at + n], md, cache, None))
        at += n
    return torch.cat(got).double(), want, wd, h.double(), m, v1


ATTENTION = [rotary(6, 2, 8, 6, 4, 30.0, 0.45, (3.0, 20, 2.0, 0.3)), rotary(3, 3, 5, 5, 0, 10.0, 0.7),
             rotary(1, 1, 6, 9, 6, 100.0, 1.0, None, None, False),
             biased(6, 2, 8, 6, 5, 0.45, 0.8, 3), biased(4, 1, 5, 12, 1, 0.7, 0.5, 1),
             biased(5, 5, 7, 3, 13, 0.4, 0.0, 2, None, False), biased(2, 2, 6, 6, 100, 0.9, 0.3, 100)]


@pytest.mark.parametrize("i", range(len(ATTENTION)))
def test_attention_layers(i):
    from vllm_gcu_b200.config import AttentionSpec
    layer, g, H, T = ATTENTION[i], gen(i), 20, 23
    m = layer["mixer"]
    width = m["kv_heads"] * m["vdim"]
    cases = [None]
    if m["v_mix"]:      # the first layer's values lie in other heads
        G = next(n for n in (5, 4, 3, 2, 1) if width % n == 0)
        cases.append((AttentionSpec(G, G, 8, 1.0, v_head_dim=width // G), rand(g, T, width)))
    for first in cases:
        for sizes in ([T], [1] * T, [9, 1, 1, 2, 10]):
            got, want, w, h, _, v1 = _attention_case(layer, first, H, T, gen(i), sizes)
            assert torch.allclose(got, want, atol=1e-5), sizes
    if layer["type"] == "attention":        # the sinks matter, and their size does
        w["sink"] = w["sink"] - 3
        assert (O.rotary_attention(h, w, m, 1e-3, v1)[0] - want).abs().max() > 1e-2


def test_mixed_values_must_fit():
    from vllm_gcu_b200.config import ModelConfig
    from vllm_gcu_b200.models import build_model
    cfg = model_config(8, 8, [biased(2, 1, 4, 4, 3, 1.0, 0.0, 1), rotary(2, 2, 4, 4, 2, 10.0, 1.0)], 1)
    with pytest.raises(ValueError, match="values mixed"):
        build_model(ModelConfig.from_hf_dict(cfg, dtype="float32"), "cpu")


@pytest.mark.parametrize("N,D,R", [(4, 6, 5), (1, 3, 1), (3, 33, 8)])
def test_time_mixing_portions_and_slots(N, D, R):
    from vllm_gcu_b200.config import TimeMixSpec
    from vllm_gcu_b200.layers.input_conv import InputConv
    from vllm_gcu_b200.layers.recurrent import TimeMix
    from vllm_gcu_b200.ops import ref
    g, T, H, taps = gen(N), 11, 10, 3
    m = TimeMix(TimeMixSpec(N, D, R), H, 1e-3, torch.float32, "cpu", "p")
    conv = InputConv(H, taps, torch.float32, "cpu", "c", m.mu)
    shapes = {k[7:]: s for k, s in O.tensor_shapes(model_config(8, H, [wkv(N, D)], 1), R).items()
              if k.startswith("l0.mix.")}
    w = {n: rand(g, *s) * (s[-1] ** -0.5 if len(s) > 1 and n != "u" else 1.0)
         for n, s in shapes.items()}
    w["w0"] = w["w0"] - 1
    assert m.tensor_names() == set(w) and all(m.load(n, t) for n, t in w.items())
    m.finalize()
    cw = rand(g, H, taps)
    conv.load_weight("weight", cw)
    h = rand(g, T, H)
    want = O.wkv_mixer(O.input_conv(h.double(), cw.double()), {n: t.double() for n, t in w.items()},
                       {"heads": N, "dim": D}, 1e-3)
    shapes = {**conv.state_shapes(), **m.state_shapes()}
    assert shapes["inputs"][0] == (taps, H) and shapes["matrix"][1] == torch.float32
    state = {k: torch.full((3, *s), 5.0) for k, (s, _) in shapes.items()}
    for sizes in SCHEDULES:                     # each leaves its state behind in the slot
        at, got = 0, []
        for n in sizes:
            md = Step([(2, at, n)], decodes=int(n == 1 and at % 2 == 0))
            mixed = torch.empty(5, n, H)
            ref.input_conv(h[at:at + n], conv.weight, m.mu, md, state["inputs"], mixed)
            got.append(m(mixed, md, state))
            at += n
        assert torch.allclose(torch.cat(got).double(), want, atol=1e-5), sizes
    assert (state["matrix"][:2] == 5.0).all()   # other slots are left alone


@pytest.mark.parametrize("E,top,groups,keep,shared", [(6, 3, 3, 2, 5), (5, 5, 1, 1, 0),
                                                      (8, 3, 2, 1, 4), (4, 1, 4, 3, 0)])
def test_experts_of_the_best_groups(E, top, groups, keep, shared):
    from vllm_gcu_b200.layers.moe import GatedSharedMoE
    from vllm_gcu_b200.ops import ref
    g, H, F, T = gen(E), 12, 7, 40
    m = GatedSharedMoE(E, top, 1.0, H, F, shared, torch.float32, "cpu", "x", act="gelu",
                       groups=(groups, keep), shared_gate=False)
    f = moe(E, top, F, shared, (groups, keep))
    shapes = {k[7:]: s for k, s in O.tensor_shapes(model_config(8, H, [wkv(1, 4, f)], 1)).items()
              if k.startswith("l0.mlp.")}
    w = {n: 2 * rand(g, *s) * s[1] ** -0.5 for n, s in shapes.items()}
    assert m.tensor_names() == set(w) and all(m.load(n, t) for n, t in w.items())
    assert not m.load("shared.sg", torch.zeros(1, H)) and not m.load(f"e{E}.up", w["e0.up"])
    h = rand(g, T, H)
    y, rows = m(h)
    s, lo = torch.empty(T, H), torch.empty(T, H)
    ref.add_group_norm(torch.zeros(T, H), y, 1.0, torch.ones(H), 1, 1e-6, lo, out=s, **rows)
    wd = {n: t.double() for n, t in w.items()}
    assert torch.allclose(s.double(), O.experts(h.double(), wd, f), atol=1e-5)
    if keep < min(groups, top):       # the groups decide somewhere
        plain, _ = O.route(h.double(), wd["router"], top, 1, 1)
        ids, _ = O.route(h.double(), wd["router"], top, groups, keep)
        assert (plain.sort(-1).values != ids.sort(-1).values).any()


def test_activations():
    from vllm_gcu_b200.ops import ref
    x = torch.linspace(-8, 8, 200).double()
    u = x.float()[None]
    assert torch.allclose(ref.ungated_act(u.clone(), "gelu")[0].double(), O.gelu_erf(x), atol=1e-6)
    assert torch.allclose(ref.act_and_mul(torch.cat([u, u], -1), "gelu_tanh")[0].double(),
                          O.gelu_tanh(x) * x, atol=1e-5)
    assert (O.gelu_erf(x) - O.gelu_tanh(x)).abs().max() > 1e-4


# -- configuration ----------------------------------------------------------------------
def test_configuration_reads_every_number():
    from vllm_gcu_b200.config import AttentionSpec, ModelConfig, TimeMixSpec
    cfg = ModelConfig.from_hf_dict(CONFIGS["uneven"], dtype="float32")
    assert (cfg.residual_mult, cfg.norm_groups, cfg.conv_taps, cfg.rms_norm_eps) == (0.7, 3, 4, 1e-4)
    specs = [s.parts[0][2] for s in cfg.layer_specs]
    assert specs[0] == TimeMixSpec(3, 12, 12)
    assert specs[1] == AttentionSpec(6, 2, 20, 0.3, v_head_dim=28, window=24, distance_bias=True,
                                     sink="zero", temp_coef=0.4, temp_every=7, v_mix=True)
    assert specs[2] == AttentionSpec(4, 4, 16, 0.31, 12, 500.0, v_head_dim=14, rot_halves=True,
                                     rot_scaling=(3.0, 64.0, 4.0, 0.25), qk_norm=True, v_norm=True,
                                     v_mix=True, sink="learnt")
    assert specs[3].rot_scaling == () and not specs[3].v_mix
    assert [s.has_mlp for s in cfg.layer_specs] == [True, True, True, False, False]
    l0 = cfg.layer_specs[0]
    assert (l0.num_experts, l0.num_experts_per_tok, l0.router_groups, l0.router_keep,
            l0.moe_intermediate_size, l0.shared_intermediate_size) == (6, 3, 3, 2, 24, 20)
    assert cfg.kv_bytes_per_token() == 4 * (2 * 48 + 4 * 30 + 48)
    for bad, msg in ((moe(6, 2, 4, 0, (4, 2)), "groups"), (moe(6, 3, 4, 0, (3, 1)), "per token"),
                     ({"kind": "other"}, "unknown feed-forward")):
        with pytest.raises(ValueError, match=msg):
            ModelConfig.from_hf_dict(model_config(8, 8, [wkv(1, 4, bad)], 1))
    with pytest.raises(ValueError, match="groups over"):
        ModelConfig.from_hf_dict(model_config(8, 8, [wkv(1, 4)], 1, 3))
    with pytest.raises(ValueError, match="unknown mixer"):
        ModelConfig.from_hf_dict(model_config(8, 8, [{**wkv(1, 4), "type": "x"}], 1))


def test_ranks_come_from_the_checkpoint(tmp_path):
    from vllm_gcu_b200.config import ModelConfig
    cfg = CONFIGS["uneven"]
    w = O.random_model(cfg, 0, ranks=11)
    path = write_checkpoint(tmp_path / "m", cfg, w)
    assert ModelConfig.from_pretrained(path).layer_specs[0].parts[0][2].decay_rank == 11
    toks = tokens_for(cfg, 20)
    got = run(replayer(path, "cpu", max_tokens=64), {"a": toks}, [[("a", 20)]])["a"]
    assert errors(got, O.forward(cfg, w, toks)).max() < TOL


def test_missing_tensors_and_bad_sizes_are_refused():
    from vllm_gcu_b200.config import ModelConfig
    from vllm_gcu_b200.models import build_model
    cfg = CONFIGS["ones"]
    w = O.random_model(cfg, 0)
    m = build_model(ModelConfig.from_hf_dict(
        cfg, dtype="float32", tensor_shapes={k: tuple(v.shape) for k, v in w.items()}), "cpu")
    del w["l0.canon1"]
    with pytest.raises(ValueError, match="missing"):
        m.load_weights(w.items())
    for layer, taps, msg in ((wkv(1, 300), 1, "keys per head"), (wkv(1, 4), 9, "taps"),
                             (rotary(3, 2, 4, 4, 2, 10.0, 1.0), 1, "key heads"),
                             (rotary(2, 2, 4, 4, 3, 10.0, 1.0), 1, "rotated"),
                             (biased(2, 2, 4, 4, 3, 1.0, 0.1, 0), 1, "temperature")):
        with pytest.raises(ValueError, match=msg):
            build_model(ModelConfig.from_hf_dict(model_config(8, 8, [layer], taps),
                                                 dtype="float32"), "cpu")


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
    cfg, w, path = build(tmp_path, "uneven", seed=4, weights=peaked_model)
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


@pytest.mark.parametrize("window", [1, 5, 16, 33])
def test_window_edges_in_prompts_and_in_decoding(tmp_path, window):
    """One windowed layer alone, one tap: a token just inside the window of the last position
    changes its logits, one just outside does not, and the engine agrees."""
    cfg = model_config(70, 24, [biased(8, 2, 12, 8, window, 0.5, 0.5, 9, None)], 1)
    w = peaked_model(cfg, window)
    path = write_checkpoint(tmp_path / "m", cfg, w)
    n = 70
    base = tokens_for(cfg, n, 1)
    before = O.forward(cfg, w, base)[-1:]
    rp = replayer(path, "cpu", max_tokens=128)
    for back in sorted({0, 1, window - 2, window - 1, window, window + 1}):
        if not 0 <= back < n:
            continue
        # of some tokens in this place the one that moves the last logits most
        swaps = [base[:n - 1 - back] + [t] + base[n - back:] for t in range(0, cfg["vocab"], 7)]
        toks = max(swaps, key=lambda x: errors(O.forward(cfg, w, x)[-1:], before).item())
        want = O.forward(cfg, w, toks)
        assert (errors(want[-1:], before) > 1e-3).item() == (back < window)
        for sizes in ([n], [n - 3, 2, 1], [n - 4, 1]):
            got = run(rp, {"a": toks}, [[("a", c)] for c in portions(n, sizes)])["a"]
            assert errors(got, want).max() < TOL, (back, sizes)
            assert (errors(got[-1:], before) > 1e-3).item() == (back < window)


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
    toks = tokens_for(cfg, 40)
    got = run(replayer(path, "cpu", max_tokens=64), {"a": toks}, [[("a", 40)]])["a"]
    assert errors(got, O.forward(cfg, w, toks)).max() < TOL
    names = ("sink_softmax", "visible", "slopes", "temperature", "frequencies", "wkv", "decays",
             "input_conv", "mix_values", "route", "gelu_erf", "gelu_tanh", "group_norm")
    real = {n: getattr(O, n) for n in names}
    wrong = {
        "sink_softmax": lambda s, sink: torch.softmax(s, -1),
        "visible": lambda T, window=None: real["visible"](T, window and window + 1),
        "slopes": lambda n: [2.0 ** (-8.0 * a / n) for a in range(n)],
        "temperature": lambda T, c, e: real["temperature"](T + 1, c, e)[1:],
        "frequencies": lambda d, b, s: (real["frequencies"](d, b, s)[0], 1.0),
        "wkv": lambda r, k, v, d, u: torch.cat([real["wkv"](r[:9], k[:9], v[:9], d[:9], u),
                                                real["wkv"](r[9:], k[9:], v[9:], d[9:], u)]),
        "decays": lambda h, lw: torch.exp(-torch.exp((h @ lw["w1"].T) @ lw["w2"].T + lw["w0"])),
        "input_conv": lambda x, t: torch.cat([real["input_conv"](x[:16], t),
                                              real["input_conv"](x[16:], t)]),
        "mix_values": lambda v, share, first: v,
        "route": lambda h, r, top, g, k: real["route"](h, r, top, 1, 1),
        "gelu_erf": real["gelu_tanh"], "gelu_tanh": real["gelu_erf"],
        "group_norm": lambda x, wt, g, eps: real["group_norm"](x, wt, 1, eps),
    }
    for name, f in wrong.items():
        setattr(O, name, f)
        try:
            assert errors(got, O.forward(cfg, w, toks)).max() > 2 * TOL, name
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
    from vllm_gcu_b200.models.vadelix import VadelixForCausalLM
    m = build_model(preset("tiny-vadelix", dtype="float32"), "cpu")
    m.init_random(0)
    assert [s is None for s in m.kv_cache_spec()["layer_shapes"]] == [False, True, False, False]
    assert m.first_mixing == 0 and m.layers[2].mix.parts[0].first is not None
    assert float(m.layers[2].mix.parts[0].share) == 0.5
    assert preset("vadelix-12b", num_hidden_layers=4).layer_specs[3].mixer == "wkv"
    assert set(VadelixForCausalLM.native_sources) <= {p.stem for p in b.CSRC.glob("*.cu")}


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
    app = build_app(eng, ByteTokenizer(mc.vocab_size), "vadelix")
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
