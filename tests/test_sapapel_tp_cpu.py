"""Sapapel over two tensor-parallel CPU ranks: heads, expert width and vocabulary sharded, latent
rows, shift state and residual stream replicated."""
import os
import socket
import sys

import pytest
import torch
import torch.distributed as dist
import torch.multiprocessing as mp

import sapapel_oracle as O
from sapapel_cases import layer, model_config, tokens_for, write_checkpoint

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CONFIG = model_config(90, 40, 1.6, 1e-5, [layer(4, 12, 20, 28, 0.3, 5, 2, 24),
                                          layer(2, 16, 8, 20, 0.25),
                                          layer(6, 8, 8, 36, 0.4, 3, 1, 12)])
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
    layer0 = llm.engine.model.layers[0]
    assert layer0.mix.N == 2 and layer0.mlp.experts.inter_real == 12
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
    want = []
    for p in PROMPTS:
        toks = list(p)
        for _ in range(6):
            toks.append(int(O.forward(CONFIG, w, toks)[-1].argmax()))
        want.append(toks[len(p):])
    torch.save(want, os.path.join(path, "want.pt"))
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
