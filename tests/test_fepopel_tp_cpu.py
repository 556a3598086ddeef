"""Fepopel over two tensor-parallel CPU ranks: heads, expert widths and vocabulary sharded, latent
rows, norms of heads, router and residual stream replicated."""
import os
import socket
import sys

import pytest
import torch
import torch.distributed as dist
import torch.multiprocessing as mp

import fepopel_oracle as O
from fepopel_cases import (chunked, dense, greedy, latent, model_config, moe, tokens_for,
                           write_checkpoint)

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CONFIG = model_config(90, 40, [latent(4, 12, 4, 20, 28, 50.0, 0.3, moe(5, 2, 24, 16, 1.5)),
                               chunked(4, 2, 12, 20, 10, 0.4, 5.0, moe(3, 1, 12)),
                               latent(2, 16, 6, 8, 20, 900.0, 0.25, dense(24))], (0, 2, 2))
PROMPTS = [tokens_for(CONFIG, n, n) for n in (1, 19, 34)]


def _worker(rank, world, port, path):
    sys.path[:0] = [ROOT, os.path.join(ROOT, "tests")]
    os.environ.update({"RANK": str(rank), "WORLD_SIZE": str(world), "LOCAL_RANK": str(rank),
                       "MASTER_ADDR": "127.0.0.1", "MASTER_PORT": str(port)})
    from vllm_gcu_b200.parallel.state import init_distributed
    init_distributed(tp=world, backend="gloo")
    from vllm_gcu_b200.engine.llm import LLM
    from vllm_gcu_b200.engine.request import SamplingParams
    llm = LLM(path, device="cpu", dtype="float32", tensor_parallel_size=world, max_num_seqs=4,
              max_num_batched_tokens=16, max_model_len=128, num_gpu_blocks=32)
    layers = llm.engine.model.layers
    assert layers[0].mix.N == 2 and layers[0].mlp.experts.inter_real == 12
    assert (layers[1].mix.parts[0].H, layers[1].mix.parts[0].G) == (2, 1)
    outs = llm.generate(PROMPTS, SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True))
    want = torch.load(os.path.join(path, "want.pt"))
    got = [o.outputs[0].token_ids for o in outs]
    assert got == want, (got, want)
    dist.barrier()
    dist.destroy_process_group()


@pytest.mark.timeout(300)
def test_tensor_parallel_generation(tmp_path):
    w = O.random_model(CONFIG, 2)
    path = write_checkpoint(tmp_path / "m", CONFIG, w)
    torch.save([greedy(CONFIG, w, p, 6) for p in PROMPTS], os.path.join(path, "want.pt"))
    with socket.socket() as s:
        s.bind(("127.0.0.1", 0))
        port = s.getsockname()[1]
    mp.spawn(_worker, args=(2, port, path), nprocs=2, join=True)


def test_layouts_without_tensor_parallel_shards_are_refused(monkeypatch):
    from vllm_gcu_b200.config import ModelConfig
    from vllm_gcu_b200.models import build_model
    from vllm_gcu_b200.parallel.state import GroupCoordinator, get_state
    cfg = ModelConfig.from_hf_dict(CONFIG, dtype="float32")
    for group in ("pp", "dp", "ep"):
        with monkeypatch.context() as m:
            m.setattr(get_state(), group, GroupCoordinator(group, [0, 1], 0))
            with pytest.raises(ValueError, match="tensor parallelism only"):
                build_model(cfg, "cpu")
