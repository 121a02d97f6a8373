"""Rank of the tensor-parallel tests of the families whose layers are configured one by one (launched by torchrun, gloo
on the CPU): its shard of a seeded model runs a prompt in two portions; rank 0 writes the logits. argv: out_path family
config_name"""
import importlib
import os
import sys

import torch
import torch.distributed as dist

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

from ksanallm_b200.config import model_config_from_hf  # noqa: E402
from ksanallm_b200.models.common import StepInput  # noqa: E402
from ksanallm_b200.models.weights import DictSource, build_model  # noqa: E402
from ksanallm_b200.parallel.comm import TPComm  # noqa: E402


def main():
    out, family, name = sys.argv[1:4]
    hlp = importlib.import_module(family + "_helpers")
    os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
    dist.init_process_group("gloo")
    rank, world = dist.get_rank(), dist.get_world_size()
    c = hlp.SPLIT.get(name) or hlp.CONFIGS[name]
    model = build_model(model_config_from_hf(c), DictSource(hlp.weights(c, 3), family), rank, world,
                        TPComm(dist.group.WORLD, rank, world, "nccl", "cpu"), device="cpu", dtype=torch.float32, max_positions=256)
    model.allocate_kv_cache(8, 16)
    t, parts, at = hlp.tokens(c, 60), [], 0
    i32 = lambda x: torch.tensor(x, dtype=torch.int32)  # noqa: E731
    with torch.inference_mode():
        for n in (45, 15):
            pos = list(range(at, at + n))
            parts.append(model.forward(StepInput(
                i32(t[at:at + n]), i32(pos), i32(pos), i32([0, n]), i32([at + n]), torch.arange(8, dtype=torch.int32).view(1, 8),
                num_multi=1, num_single=0, num_tokens=n, num_multi_tokens=n, max_q_len=n, max_kv_len=at + n,
                prev_ids=i32([t[p - 1] if p else -1 for p in pos]))))
            at += n
    logits = torch.cat(parts)
    others = [torch.empty_like(logits) for _ in range(world)]
    dist.all_gather(others, logits)
    assert all(torch.equal(o, logits) for o in others)
    if rank == 0:
        torch.save(logits, out)
    dist.destroy_process_group()


if __name__ == "__main__":
    main()
