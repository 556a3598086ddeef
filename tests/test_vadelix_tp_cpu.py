"""Vadelix over two tensor-parallel CPU ranks: heads, states, experts and vocabulary sharded,
norms over whole projections across ranks."""
import os
import socket
import sys

import pytest
import torch
import torch.distributed as dist
import torch.multiprocessing as mp

import vadelix_oracle as O
from vadelix_cases import (biased, dense, greedy, model_config, moe, rotary, tokens_for, wkv,
                           write_checkpoint)

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CONFIG = model_config(90, 40, [
    biased(4, 2, 12, 10, 9, 0.3, 0.5, 6, dense(24)),
    wkv(4, 8, moe(6, 2, 12, 20, (3, 2))),
    rotary(8, 4, 16, 5, 8, 100.0, 0.3, (2.0, 50, 4.0, 0.5), moe(4, 2, 8)),
    wkv(2, 20)], 3, 4, 0.7)
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
    first, last = layers[0].mix.parts[0], layers[2].mix.parts[0]
    assert first.H == 2 and layers[1].mix.N == 2 and last.q_norm.shape == (4 * 16,)
    slopes = torch.tensor([2.0 ** (-2.0 * (2 * rank + h + 1)) for h in range(2)])
    assert torch.allclose(first.slopes, slopes)
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


def test_layouts_that_cannot_be_sharded_are_refused(monkeypatch):
    from vllm_gcu_b200.config import ModelConfig
    from vllm_gcu_b200.models import build_model
    from vllm_gcu_b200.parallel.state import GroupCoordinator, get_state
    cfg = ModelConfig.from_hf_dict(CONFIG, dtype="float32")
    for group in ("pp", "dp", "ep"):
        with monkeypatch.context() as m:
            m.setattr(get_state(), group, GroupCoordinator(group, [0, 1], 0))
            with pytest.raises(ValueError, match="tensor parallelism only"):
                build_model(cfg, "cpu")
    for layer in (wkv(3, 4), rotary(4, 1, 4, 4, 2, 10.0, 1.0), biased(3, 3, 4, 4, 2, 1.0, 0.0, 1)):
        odd = ModelConfig.from_hf_dict(model_config(8, 8, [layer], 1), dtype="float32")
        with monkeypatch.context() as m:
            m.setattr(get_state(), "tp", GroupCoordinator("tp", [0, 1], 0))
            with pytest.raises(ValueError, match="over 2 ranks"):
                build_model(odd, "cpu")
