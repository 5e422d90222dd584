"""CPU tests of the Migosun family: the oracle's own consistency, configuration and checkpoint handling, and the engine's
host code on gloo ranks with stand-in ops."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import migosun_util as mu
from oracle import migosun_oracle as mo

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("world", [1, 2])
def test_engine_on_cpu_ranks(world):
    cmd = [sys.executable, "-m", "torch.distributed.run", "--nnodes=1", f"--nproc-per-node={world}", "--master-addr", "127.0.0.1",
           "--master-port", str(29770 + world), os.path.join(ROOT, "tests", "layers_cpu_worker.py"), "migosun"]
    env = dict(os.environ, OMP_NUM_THREADS="2", CUDA_VISIBLE_DEVICES="")
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=600, env=env)
    assert r.returncode == 0, r.stdout[-3000:] + r.stderr[-3000:]
    assert "LAYERS-CPU-OK" in r.stdout


def test_oracle_mechanisms_by_hand():
    # the first two of three dimensions turn by one radian
    x = torch.tensor([[[1.0, 2.0, 5.0]]], dtype=torch.float64)
    got = mo.rotate_first_dims(x, torch.tensor([1]), 2, 7.0)
    c, s = torch.cos(torch.tensor(1.0, dtype=torch.float64)), torch.sin(torch.tensor(1.0, dtype=torch.float64))
    assert torch.allclose(got, torch.stack([c - 2 * s, 2 * c + s, torch.tensor(5.0, dtype=torch.float64)]).view(1, 1, 3))
    m = mo.chunk_mask(7, 3)
    assert m.sum(-1).tolist() == [1, 2, 3, 1, 2, 3, 1] and m[4].tolist() == [False, False, False, True, True, False, False]
    p = mo.softmax_with_sink(torch.tensor([[[0.0, float("-inf")]]]), torch.tensor([0.0]))
    assert torch.allclose(p, torch.tensor([[[0.5, 0.0]]]))  # one key and the sink share the weight
    y = mo.short_conv(torch.tensor([[1.0], [10.0], [100.0]]), torch.tensor([[2.0, 3.0]]))
    assert y.view(-1).tolist() == [3.0, 32.0, 320.0]  # the last column multiplies the current token
    # one channel: decay 0.5, then u = beta (v - S k), S += k u, read with the write seen
    o, st = mo.delta_recurrence(*(torch.tensor(v).view(2, 1, 1) for v in ([1.0, 1.0], [1.0, 2.0], [4.0, 7.0], [0.5, 0.5])), torch.tensor([[0.5], [1.0]]))
    # t0: S = 0.5 * 4 = 2; t1: S = 1, u = 7 - 2 = 5, S = 1 + 10 = 11
    assert o.view(-1).tolist() == [2.0, 11.0] and st.item() == 11.0
    o, st = mo.linear_attention_recurrence(*(torch.tensor(v).view(2, 1, 1) for v in ([1.0, 3.0], [1.0, 2.0], [4.0, 7.0], [0.5, 0.5])))
    assert o.view(-1).tolist() == [4.0, 48.0] and st.item() == 16.0
    g = mo.delta_decay(torch.tensor([[[0.0]]]), torch.tensor([0.0]), torch.tensor([0.0]))
    assert torch.allclose(g, torch.tensor(0.5))  # exp(-log 2)
    a, b = torch.tensor([[[1.0]], [[10.0]]]), torch.tensor([[0.5, 2.0], [0.25, 1.0]])
    new = mo.join_streams(a, torch.tensor([1.0, 0.1]), b, torch.tensor([1.0, -1.0]), lambda u: u)
    assert new.view(-1).tolist() == [0.5 + 2.5 + 2.0, 2.0 + 10.0 - 2.0]


def test_oracle_is_causal_and_chunked():
    """Changing a token changes nothing before it; with the recurrence's output off, nothing past its chunk."""
    case = mu.config(32, 50, 2, [(mu.side_by_side((2, 1, 8, 8, 6, 4, 1e4, 0.4), (1, 1, 4, 4, 3, (2, 2))), mu.dense(8))])
    cfg, w = case[0], mu.weights(case, 1)
    a = mu.tokens(cfg, 30)
    b = a.clone()
    b[13] = (b[13] + 1) % 50
    d = (mu.reference(cfg, w, a, torch.float64) - mu.reference(cfg, w, b, torch.float64)).abs().amax(-1)
    assert d[:13].max() == 0 and d[13] > 1e-3 and d[25] > 1e-7  # the state carries it on
    w["l0.mix.right.o"].zero_()
    d = (mu.reference(cfg, w, a, torch.float64) - mu.reference(cfg, w, b, torch.float64)).abs().amax(-1)
    assert d[13:18].min() > 1e-6 and d[18:].max() == 0


def test_model_class_and_ranks_from_the_checkpoint(tmp_path):
    from gpt_fast import gpt_migosun_TP, loader
    case = mu.CONFIGS["uneven"]
    cfg, w = case[0], mu.weights(case, 2)
    mu.save(cfg, w, tmp_path)
    cls, args = loader.model_class(str(tmp_path))
    assert cls is gpt_migosun_TP.GPTMigosun and args.n_layer == 4 and args.dim == 92 and args.streams == 3 and torch.float32 in cls.dtypes
    assert args.embed_scale == 0.7
    right = args.layers[0]["mixer"]["right"]
    assert (right["decay_rank"], right["gate_rank"]) == (5, 9) and args.layers[1]["mixer"]["decay_rank"] == 6
    assert "decay_rank" not in json.load(open(tmp_path / "config.json"))["layers"][0]["mixer"]["right"]


def test_bad_configurations_are_refused():
    from gpt_fast import mixers
    good = mu.side_by_side((4, 2, 8, 8, 5, 4, 1e4, 1.0), (2, 1, 4, 4, 2, (2, 2)))["mixer"]

    def broken(side, **kw):
        m = copy.deepcopy(good)
        m["right"].update(decay_rank=2, gate_rank=2)
        m[side].update(kw)
        return m

    mixers.make_mixer("parallel", 8, broken("left"))
    for side, kw, text in (("left", dict(kv_heads=3), "evenly"), ("left", dict(rot={"base": 1e4, "dims": 3}), "rotated"),
                           ("left", dict(rot={"base": 1e4, "dims": 10}), "rotated"), ("right", dict(heads=3, kv_heads=2), "evenly"),
                           ("right", dict(conv=0), "taps"), ("left", dict(mask={"size": -1}), "chunk")):
        with pytest.raises(ValueError, match=text):
            mixers.make_mixer("parallel", 8, broken(side, **kw))


def test_checkpoint_round_trip_and_missing_tensor(tmp_path):
    from gpt_fast import loader
    case = mu.CONFIGS["uneven"]
    cfg, w = case[0], mu.weights(case, 2)
    mu.save(cfg, w, tmp_path)
    model = loader.load_model(str(tmp_path), torch.bfloat16, "cpu")
    assert model.output.weight is model.tok_embeddings.weight and torch.equal(model.output.weight, w["embed"])
    b, m = model.layers[0].mixer, model.layers[0].mixer.sublayer
    at, rows = 0, b.in_proj.weight
    for name, pad in (("left.q", 0), ("left.k", 0), ("left.v", 0), ("right.q", 0), ("right.k", 0), ("right.v", 0), ("right.a1", 3), ("right.g1", 7), ("right.b", 0)):
        t = w["l0.mix." + name]
        assert torch.equal(rows[at:at + t.shape[0]], t) and rows[at + t.shape[0]:at + t.shape[0] + pad].abs().sum() == 0, name
        at += t.shape[0] + pad
    assert rows[at:].abs().sum() == 0 and rows.shape[0] % 8 == 0
    assert torch.equal(m.right.a2[:, :5], w["l0.mix.right.a2"]) and m.right.a2.shape[1] == 8 and m.right.a2[:, 5:].abs().sum() == 0
    assert torch.equal(m.wo.weight, torch.cat([w["l0.mix.left.o"], w["l0.mix.right.o"]], 1))
    assert torch.equal(b.w_mix, w["l0.hc1.mix"]) and torch.equal(model.layers[0].mlp.w_in, w["l0.hc2.in"])
    assert torch.equal(model.layers[0].mlp.sublayer.w1, torch.cat([w["l0.mlp.up"], w["l0.mlp.gate"]])) and model.layers[1].mlp is None
    del w["l2.mix.right.A_log"]
    mu.save(cfg, w, tmp_path)
    with pytest.raises(KeyError):
        loader.load_model(str(tmp_path), torch.bfloat16, "cpu")


def test_presets_build_with_one_embedding_table():
    from gpt_fast import gpt_migosun_TP as mg
    for name in mg.transformer_configs:
        with torch.device("meta"):
            model = mg.GPTMigosun.from_name(name)
        assert len(model.layers) == model.config.n_layer
        assert "output.weight" not in dict(model.named_parameters())
    kinds = [b.mixer.sublayer.kind for b in model.layers]
    assert kinds[:3] == ["parallel", "parallel", "gla"]
    model = mg.GPTMigosun.from_name("migosun-tiny").to(torch.bfloat16)
    assert model.output.weight is model.tok_embeddings.weight and model.output.weight.dtype == torch.bfloat16


def test_entry_points_check_arguments_without_a_gpu():
    from gpt_fast import _C
    lib = _C.lib
    assert lib.lri_join_streams(0, 16, 16, 16, 16, 16, 16, 16, 1e-5, 16, 1, 17, 8, None) == -3 and b"streams" in lib.lri_last_error()
    assert lib.lri_join_streams(0, None, 16, 16, 16, 16, 16, 16, 1e-5, 16, 1, 4, 8, None) == -1
    assert lib.lri_gateup_glu(2, 16, 16, 16, 4, 8, 8, 1.7, 1.0, 1.0, None, 0, None) == -5
    assert lib.lri_gateup_glu_workspace_bytes(2, 4, 8, 8) == 4 * 16 * 4 and lib.lri_gateup_glu_workspace_bytes(0, 500, 64, 64) == 0
    assert lib.lri_grouped_attention(0, 16, 16, 16, None, 16, 8, 1.0, 16, 0, 8, 0, 0, 1.0, 1, 1, 3, 2, 8, 8, None) == -1
    assert lib.lri_state_scan(16, 16, 16, 16, 16, 16, 8, 16, 16, 0, 16, 1, 1, 1, 600, 8, None) == -3
    assert lib.lri_state_blocks(1) == 1 and lib.lri_state_blocks(9) == 3
    assert lib.lri_state_step_supports(128, 128, 16, 16) == 1 and lib.lri_state_step_supports(300, 8, 8, 8) == 0
    assert lib.lri_state_step_supports(64, 64, 12, 8) == 0
    assert lib.lri_head_norm_gate(0, 16, 16, 1e-5, 16, 8, 2, 1.0, 16, 8, 1, 1, 8, None) == -1
