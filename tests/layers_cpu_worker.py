"""One gloo rank of the layer-engine test (started by tests/test_patevik_cpu.py through torch.distributed.run): the
Patevik engine with the CPU stand-in ops against the oracle, whole prompts, portions, single tokens, batches and reused
rows, heads and expert widths split over the ranks."""
import os
import sys

import torch
import torch.distributed as dist

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(HERE)
for p in (HERE, ROOT, os.path.join(ROOT, "ladder-residual-inference_b200")):
    sys.path.insert(0, p)

dist.init_process_group("gloo")

import patevik_util as pu  # noqa: E402
from cpu_layer_ops import CpuLayerOps  # noqa: E402

world = dist.get_world_size()
cfg = pu.config(48, 61, [(pu.recurrent(2, 6, 8), pu.experts(4, 2, 12)), (pu.latent(4, 6, 4, 10, 12, 9), pu.experts(3, 3, 8)),
                         (pu.latent(2, 8, 2, 6, 8, 30), None), (pu.recurrent(4, 4, 6), pu.experts(5, 1, 8))])
w = pu.weights(cfg, 3)
model = pu.build(cfg, w, torch.float32, "cpu", 2, 64)
model._engine.ops = CpuLayerOps
seqs = torch.stack([pu.tokens(cfg, 41, 5), pu.tokens(cfg, 41, 6)])
ref = torch.stack([pu.reference(cfg, w, s) for s in seqs])
for cuts in ([41], [1], [2, 3, 5, 1], [30, 1], [8, 9]):
    got = pu.feed(model, seqs, cuts, device="cpu")
    assert pu.row_err(got, ref).max() < 2e-5, (cuts, pu.row_err(got, ref).max())
# a row used again for another sequence, alone
other = pu.tokens(cfg, 23, 9)
got = pu.feed(model, other[None], [7, 1, 1, 5], device="cpu")
assert pu.row_err(got[0], pu.reference(cfg, w, other)).max() < 2e-5
# greedy through the head that is split by vocabulary
pu.feed(model, seqs[:, :20], [20], device="cpu")
tok = model.decode_greedy(seqs[:, 20:21].int(), torch.tensor([20], dtype=torch.int32))
assert torch.equal(tok.view(-1).long(), ref[:, 20].argmax(-1))
if dist.get_rank() == 0:
    print("LAYERS-CPU-OK", world)
dist.destroy_process_group()
