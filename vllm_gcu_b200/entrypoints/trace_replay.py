"""Replays a trace of token ids through a model step by step and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Nothing is generated: the steps come from standard input, one JSON object a line,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` are the next tokens of each request, all of one step in one batch; ``want`` names the
places among them whose logits are written (``OUT/<step>.f32``, little-endian fp32 ``[wanted,
vocab]`` in the order of the entries); ``end`` lists the requests that are over after the step.
``done <step>`` is printed after every step.  The engine behind it is the serving engine: its
model registry, loader, block manager, batch layout, model runner and kernels, decode steps
through its CUDA graphs.  The cache holds ``N`` tokens (each request rounded up to whole blocks)
and there are four request slots, so blocks are used again.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Sequence

import torch

from ..config import CacheConfig, EngineConfig, ModelConfig, SchedulerConfig
from ..engine.llm import LLMEngine, check_token_ids
from ..engine.request import Request, SamplingParams

MAX_LIVE = 4
BLOCK_SIZE = 16


class TraceReplayer:
    def __init__(self, engine: LLMEngine):
        self.engine = engine
        self.live: dict[str, Request] = {}

    def step(self, entries: Sequence[dict], end: Sequence[str] = ()) -> torch.Tensor:
        """Runs one step; returns the wanted logits ``[wanted, vocab]`` (fp32, host)."""
        eng, vocab = self.engine, self.engine.cfg.model.vocab_size
        portions, wanted = [], []
        if len({e["id"] for e in entries}) != len(entries):
            raise ValueError("a request appears twice in a step")
        for e in entries:
            rid, toks, want = str(e["id"]), [int(t) for t in e["tokens"]], e.get("want") or []
            check_token_ids(toks, vocab)
            if any(not 0 <= w < len(toks) for w in want):
                raise ValueError(f"{rid}: wanted places {want} of {len(toks)} tokens")
            req = self.live.get(rid)
            if req is None:
                req = self.live[rid] = Request(rid, [], SamplingParams(
                    max_tokens=1 << 30, ignore_eos=True))
            req.prompt_token_ids.extend(toks)
            if req.num_prompt_tokens > eng.cfg.scheduler.max_model_len:
                raise ValueError(f"{rid}: longer than {eng.cfg.scheduler.max_model_len} tokens")
            portions.append((req, len(toks), list(want)))
            wanted.append((rid, len(want)))
        out = torch.empty(0, vocab)
        if portions:
            so = eng.scheduler.schedule_portions(portions)
            if so.total_tokens > eng.runner.max_tokens:
                raise ValueError(f"a step of {so.total_tokens} tokens, at most "
                                 f"{eng.runner.max_tokens}")
            handle = eng.runner.execute(so)
            handle.wait()                  # ids that a decode step has sampled are not looked at
            logits = handle.extra.get("logits")
            if logits is not None:
                out = torch.cat([logits[rid] for rid, n in wanted if n]).cpu()
        for rid in end:
            if self.live.pop(str(rid), None) is not None:
                eng.scheduler.abort_request(str(rid))
        return out


def build_engine(model_dir: str, dtype: str, max_tokens: int, device: str = "cuda") -> LLMEngine:
    n = -(-max_tokens // 64) * 64
    mc = ModelConfig.from_pretrained(model_dir, dtype=dtype)
    mc.max_position_embeddings = max(mc.max_position_embeddings, n)
    return LLMEngine(EngineConfig(
        model=mc, device=device, load_format="safetensors", model_path=model_dir,
        cache=CacheConfig(block_size=BLOCK_SIZE, num_gpu_blocks=n // BLOCK_SIZE,
                          enable_prefix_caching=False),
        scheduler=SchedulerConfig(max_num_seqs=MAX_LIVE, max_num_batched_tokens=n,
                                  max_model_len=n),
        cuda_graph_sizes=[1, 2, MAX_LIVE], additional_config={"keep_graph_logits": True}))


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__,
                                 formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="most tokens that live requests hold together")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"],
                    help="cpu: the torch formulation of every op (debugging)")
    args = ap.parse_args(argv)
    if args.device == "cuda":
        if not torch.cuda.is_available():
            raise SystemExit("no CUDA device")
        prepare_kernels(args.model)
    replay = TraceReplayer(build_engine(args.model, args.dtype, args.max_tokens, args.device))
    from ..ops import _native
    with torch.inference_mode():
        for line in sys.stdin:
            if not line.strip():
                continue
            job = json.loads(line)
            logits = replay.step(job.get("entries") or [], job.get("end") or [])
            if args.device == "cuda":
                _native.check_status()
            if logits.shape[0]:
                path = os.path.join(args.out, f"{job['step']}.f32")
                with open(path, "wb") as f:
                    f.write(logits.numpy().astype("<f4").tobytes())
            print(f"done {job['step']}", flush=True)
    return 0


def prepare_kernels(model_dir: str) -> None:
    """Builds the native library where it is missing or stale: the kernels of the model's family
    if it names them, else all of them."""
    from ..csrc import build
    from ..models import get_model_class
    from ..ops import _native
    if os.environ.get("VLLM_B200_NATIVE_LIB"):
        return
    arch = ModelConfig.from_pretrained(model_dir).architecture
    sources = getattr(get_model_class(arch), "native_sources", None)
    if sources is None:
        build.build()
        return
    path, partial = build.ensure(sources)
    if partial:
        _native.use_partial_library(path)


if __name__ == "__main__":
    sys.exit(main())
