"""Prefill and decode throughput of one model family beside the closest other one at equal layer
sizes, both through ``LLM.generate`` with random weights.

* Sapapel beside DeepSeek (latent attention over a paged latent cache, routed experts): same width,
  heads, latent rank, experts, experts per token, expert width, layers and vocabulary; DeepSeek's
  rows have 64 rotary columns more and it has neither the output gate nor the depth average.
* Fizunex beside Llama (grouped-query attention, dense feed-forward): same width, heads, head
  dimension, feed-forward, layers and vocabulary.  Half of Fizunex's layers are gated delta layers
  (full query / key heads), the others run attention with Llama's heads and a matrix memory.
* Fepopel beside DeepSeek: same width, heads, head and rotary dimensions, latent rank, experts,
  experts per token, expert width (routed and shared) and vocabulary; as many layer runs as DeepSeek
  has layers, two of them a second pass of a loop.  Every second layer of Fepopel has chunked grouped
  attention in place of latent attention; its experts have two matrices, DeepSeek's three.
* Vadelix beside Fizunex: same width, heads, key heads, head dimension, feed-forward, layers and
  vocabulary.  Half of the layers of both are recurrent; the others of Vadelix run attention alone, in
  turn over all keys and over a window.  Vadelix with experts beside Fepopel: same width, heads, key
  heads, experts, experts per token and expert width (routed and shared), as many layers as Fepopel has
  layer runs.

Timed on the device: the CUDA events that bracket every engine step.  Prefill: ``prompts x
input_len`` tokens in steps of 8192, one output token.  Decode: the steps of ``batch`` requests
behind a prompt of ``input_len``.

    python bench.py --workload fizunex                    (all sizes, one JSON line each)
    python benchmarks/bench_family_pair.py --pair sapapel --sizes 2048 --no-decode
"""
from __future__ import annotations

import argparse
import gc
import json
import os
import sys

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

#: per pair, width -> heads, head dims, latent rank, experts, experts per token, expert width,
#: layers; or heads, key heads, head dims, memory heads and dims, feed-forward, layers
SIZES = {"sapapel": {
    2048: dict(heads=16, dim=128, rank=512, experts=64, top=6, ff=1408, layers=8),
    4096: dict(heads=32, dim=128, rank=512, experts=32, top=4, ff=1536, layers=6),
    7168: dict(heads=128, dim=128, rank=512, experts=64, top=8, ff=2048, layers=3),
}, "fizunex": {
    2048: dict(heads=16, kv_heads=4, dim=128, mem_heads=4, mem_dim=128, mem_vdim=256, ff=8192,
               layers=8),
    4096: dict(heads=32, kv_heads=8, dim=128, mem_heads=8, mem_dim=128, mem_vdim=256, ff=14336,
               layers=8),
    8192: dict(heads=64, kv_heads=8, dim=128, mem_heads=16, mem_dim=128, mem_vdim=256, ff=28672,
               layers=4),
}, "fepopel": {
    2048: dict(heads=16, kv_heads=4, dim=128, rank=512, chunk=512, experts=64, top=6, ff=1408,
               layers=8),
    4096: dict(heads=32, kv_heads=8, dim=128, rank=512, chunk=512, experts=32, top=4, ff=1536,
               layers=6),
    7168: dict(heads=128, kv_heads=8, dim=128, rank=512, chunk=512, experts=64, top=8, ff=2048,
               layers=4),
}, "vadelix": {
    2048: dict(heads=16, kv_heads=4, dim=128, window=512, rank=64, mem_heads=4, mem_dim=128,
               mem_vdim=256, ff=8192, layers=8),
    4096: dict(heads=32, kv_heads=8, dim=128, window=512, rank=64, mem_heads=8, mem_dim=128,
               mem_vdim=256, ff=14336, layers=8),
    8192: dict(heads=64, kv_heads=8, dim=128, window=512, rank=64, mem_heads=16, mem_dim=128,
               mem_vdim=256, ff=28672, layers=4),
}, "vadelix-experts": {
    2048: dict(heads=16, kv_heads=4, dim=128, window=512, rank=512, chunk=512, experts=64, top=6,
               ff=1408, layers=8),
    4096: dict(heads=32, kv_heads=8, dim=128, window=512, rank=512, chunk=512, experts=32, top=4,
               ff=1536, layers=8),
}}
PAIRS = {"sapapel": ("sapapel", "deepseek"), "fizunex": ("fizunex", "llama"),
         "fepopel": ("fepopel", "deepseek"), "vadelix": ("vadelix", "fizunex"),
         "vadelix-experts": ("vadelix", "fepopel")}
VOCAB = 32768


def model_config(pair: str, family: str, width: int):
    from vllm_gcu_b200.config import ModelConfig
    s = SIZES[pair][width]
    if family == "fizunex":
        from vllm_gcu_b200.config import _fizunex_mixers, _fizunex_preset
        mixers = _fizunex_mixers(s["heads"], s["kv_heads"], s["dim"], s["mem_heads"],
                                 s["mem_dim"], s["mem_vdim"])
        return ModelConfig.from_hf_dict(_fizunex_preset(
            ("dp" * s["layers"])[:s["layers"]], VOCAB, width, s["ff"], *mixers), dtype="bfloat16")
    if family == "vadelix":
        from vllm_gcu_b200.config import _vadelix_preset
        e = "experts" in s
        kinds = ("we", "re", "we", "be") if e else ("wd", "rd", "wd", "bd")
        return ModelConfig.from_hf_dict(_vadelix_preset(
            " ".join((kinds * s["layers"])[:s["layers"]]), VOCAB, width, s["heads"], s["kv_heads"],
            s["dim"], s["window"], s["heads"], s["dim"], s["ff"], s.get("experts", 0),
            s.get("top", 0), (4, 2), s["ff"], s["ff"], 64), dtype="bfloat16")
    if family == "llama":
        return ModelConfig(
            architecture="LlamaForCausalLM", vocab_size=VOCAB, hidden_size=width,
            intermediate_size=s["ff"], num_hidden_layers=s["layers"],
            num_attention_heads=s["heads"], num_key_value_heads=s["kv_heads"],
            head_dim=s["dim"], tie_word_embeddings=True, dtype="bfloat16")
    if family == "fepopel":
        from vllm_gcu_b200.config import _fepopel_preset
        n = s["layers"] - 2                # the loop runs two layers once more
        return ModelConfig.from_hf_dict(_fepopel_preset(
            " ".join(("le", "ce")[i % 2] for i in range(n)), (0, 2, 2), VOCAB, width, s["heads"],
            s["dim"], 64, s["rank"], s["kv_heads"], s["chunk"], 0, s["experts"], s["top"], s["ff"],
            s["ff"]), dtype="bfloat16")
    if family == "sapapel":
        layer = {"type": "latent_attention",
                 "mixer": {"heads": s["heads"], "dim": s["dim"], "vdim": s["dim"],
                           "kv_rank": s["rank"], "scale": s["dim"] ** -0.5},
                 "mlp": {"kind": "moe", "router": {"experts": s["experts"], "top": s["top"]},
                         "expert": {"ff": s["ff"]}}}
        return ModelConfig.from_hf_dict(
            {"architecture": "Sapapel", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6},
             "postln_alpha": 2.0, "layers": [layer] * s["layers"]}, dtype="bfloat16")
    shared = pair == "fepopel"
    return ModelConfig(
        architecture="DeepseekV2ForCausalLM", vocab_size=VOCAB, hidden_size=width,
        intermediate_size=s["ff"], num_hidden_layers=s["layers"],
        num_attention_heads=s["heads"], num_key_value_heads=s["heads"], q_lora_rank=0,
        kv_lora_rank=s["rank"], qk_nope_head_dim=s["dim"], qk_rope_head_dim=64,
        v_head_dim=s["dim"], head_dim=s["dim"] + 64, num_experts=s["experts"],
        num_experts_per_tok=s["top"], moe_intermediate_size=s["ff"],
        num_shared_experts=int(shared), first_k_dense_replace=0,
        scoring_func="softmax" if shared else "sigmoid", norm_topk_prob=shared,
        rope_is_neox=False, dtype="bfloat16")


def measure(pair: str, family: str, width: int, prompts: int, input_len: int, batch: int, output_len: int,
            warmup: int, steps: int, decode: bool = True, profile: str | None = None) -> dict:
    import torch
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    from vllm_gcu_b200.ops import _native
    n = max(prompts, batch)
    llm = LLM(model_config(pair, family, width), max_num_seqs=n, max_num_batched_tokens=8192,
              max_model_len=input_len + output_len + 16, async_scheduling=True,
              enable_prefix_caching=False, cuda_graph_sizes=[batch],
              num_gpu_blocks=n * (-(-(input_len + output_len) // 16) + 2))
    eng = llm.engine
    g = torch.Generator().manual_seed(0)

    def one_pass(count: int, out_len: int, kind: str) -> tuple[int, float]:
        ids = torch.randint(0, VOCAB, (count, input_len), generator=g).tolist()
        eng.runner.timing_events, eng.runner.timing_meta = [], []
        llm.generate(ids, SamplingParams(max_tokens=out_len, temperature=0.0, ignore_eos=True))
        torch.cuda.synchronize()
        tok, ms = 0, 0.0
        for (a, b), (nd, npf, nt) in zip(eng.runner.timing_events, eng.runner.timing_meta):
            if (npf == 0 and nd == count) if kind == "decode" else nd == 0:
                tok += nt
                ms += a.elapsed_time(b)
        return tok, ms

    def timed(count: int, out_len: int, kind: str) -> float:
        for _ in range(warmup):
            one_pass(count, out_len, kind)
        tok, ms = 0, 0.0
        for _ in range(steps):
            t, m = one_pass(count, out_len, kind)
            tok, ms = tok + t, ms + m
        return tok / (ms / 1e3)

    res = {"prefill_tok_s": round(timed(prompts, 1, "prefill"), 1)}
    if decode:
        res["decode_tok_s"] = round(timed(batch, output_len, "decode"), 1)
    if profile:
        from torch.profiler import ProfilerActivity, profile as prof
        for kind, args in (("prefill", (prompts, 1)), ("decode", (batch, 8))):
            with prof(activities=[ProfilerActivity.CUDA]) as p:
                one_pass(*args, kind)
            with open(f"{profile}_{family}_{width}_{kind}.txt", "w") as f:
                f.write(p.key_averages().table(sort_by="cuda_time_total", row_limit=40,
                                               max_name_column_width=90))
    _native.check_status()
    del llm, eng
    gc.collect()
    torch.cuda.empty_cache()
    return res


def main(argv=None) -> None:
    ap = argparse.ArgumentParser(description=__doc__,
                                 formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--pair", default="fizunex", choices=sorted(PAIRS))
    ap.add_argument("--sizes", type=int, nargs="*", default=None)
    ap.add_argument("--prompts", type=int, default=16)
    ap.add_argument("--input-len", type=int, default=1024)
    ap.add_argument("--batch", type=int, default=64)
    ap.add_argument("--output-len", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--steps", type=int, default=3)
    ap.add_argument("--families", nargs="*", default=None)
    ap.add_argument("--no-decode", action="store_true")
    ap.add_argument("--profile", default=None, metavar="PREFIX",
                    help="also write a kernel table per family and phase (numbers under a "
                         "profiler: for shares only)")
    a = ap.parse_args(argv)
    for width in a.sizes or sorted(SIZES[a.pair]):
        line = {"metric": "prefill and decode tok/s, device time", "unit": "tok/s", "n_gpus": 1,
                "dtype": "bf16", "data": "synthetic (random ids, random weights)",
                "config": {"width": width, **SIZES[a.pair][width], "vocab": VOCAB, "prompts": a.prompts,
                           "input_len": a.input_len, "decode_batch": a.batch,
                           "output_len": a.output_len,
                           "l2_policy": "weights and cache larger than L2"}}
        for fam in a.families or PAIRS[a.pair]:
            line[fam] = measure(a.pair, fam, width, a.prompts, a.input_len, a.batch, a.output_len,
                                a.warmup, a.steps, not a.no_decode, a.profile)
        print(json.dumps(line), flush=True)


if __name__ == "__main__":
    main()
