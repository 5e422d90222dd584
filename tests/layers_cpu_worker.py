"""One gloo rank of the layer-engine test (started by tests/test_patevik_cpu.py and tests/test_migosun_cpu.py through
torch.distributed.run): the engine with the CPU stand-in ops against the family's oracle, whole prompts, portions, single tokens, batches and reused
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

import migosun_util as mu  # noqa: E402
import patevik_util as pu  # noqa: E402
from cpu_layer_ops import CpuLayerOps  # noqa: E402

world = dist.get_world_size()
if sys.argv[1] == "patevik":
    util = pu
    cfg = pu.config(48, 61, [(pu.recurrent(2, 6, 8), pu.experts(4, 2, 12)), (pu.latent(4, 6, 4, 10, 12, 9), pu.experts(3, 3, 8)),
                             (pu.latent(2, 8, 2, 6, 8, 30), None), (pu.recurrent(4, 4, 6), pu.experts(5, 1, 8))])
    w = pu.weights(cfg, 3)
else:
    util = mu
    case = mu.config(48, 61, 3, [(mu.side_by_side((4, 2, 6, 10, 9, 4, 500.0, 0.4), (4, 2, 6, 8, 3, (5, 9))), mu.dense(12)), (mu.linear(2, 6, 8, 4.0, 3), None),
                                 (mu.side_by_side((2, 2, 8, 6, 30, 8, 1e4, 0.3), (2, 2, 8, 4, 4, (8, 2)), (1.0, 0.4)), mu.dense(16, 0.5))])
    cfg, w = case[0], mu.weights(case, 3)
model = util.build(cfg, w, torch.float32, "cpu", 2, 64)
model._engine.ops = CpuLayerOps
seqs = torch.stack([util.tokens(cfg, 41, 5), util.tokens(cfg, 41, 6)])
ref = torch.stack([util.reference(cfg, w, s) for s in seqs])
for cuts in ([41], [1], [2, 3, 5, 1], [30, 1], [8, 9]):
    got = util.feed(model, seqs, cuts, device="cpu")
    assert util.row_err(got, ref).max() < 2e-5, (cuts, util.row_err(got, ref).max())
# a row used again for another sequence, alone
other = util.tokens(cfg, 23, 9)
got = util.feed(model, other[None], [7, 1, 1, 5], device="cpu")
assert util.row_err(got[0], util.reference(cfg, w, other)).max() < 2e-5
# greedy through the head that is split by vocabulary
util.feed(model, seqs[:, :20], [20], device="cpu")
tok = model.decode_greedy(seqs[:, 20:21].int(), torch.tensor([20], dtype=torch.int32))
assert torch.equal(tok.view(-1).long(), ref[:, 20].argmax(-1))
if dist.get_rank() == 0:
    print("LAYERS-CPU-OK", world)
dist.destroy_process_group()
