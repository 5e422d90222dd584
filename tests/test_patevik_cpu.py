"""CPU tests of the Patevik family: the oracle's own consistency, configuration and checkpoint handling, and the engine's
host code on gloo ranks with stand-in ops."""
import json
import os
import subprocess
import sys

import pytest
import torch

import patevik_util as pu
from oracle import patevik_oracle as po

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("world", [1, 2])
def test_engine_on_cpu_ranks(world):
    cmd = [sys.executable, "-m", "torch.distributed.run", "--nnodes=1", f"--nproc-per-node={world}", "--master-addr", "127.0.0.1",
           "--master-port", str(29760 + world), os.path.join(ROOT, "tests", "layers_cpu_worker.py"), "patevik"]
    env = dict(os.environ, OMP_NUM_THREADS="2", CUDA_VISIBLE_DEVICES="")
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=600, env=env)
    assert r.returncode == 0, r.stdout[-3000:] + r.stderr[-3000:]
    assert "LAYERS-CPU-OK" in r.stdout


def test_oracle_mechanisms_by_hand():
    x = torch.tensor([[3.0, 4.0]])
    assert torch.allclose(po.rms_norm(x, torch.tensor([1.0, 2.0]), 0.0), x / (12.5 ** 0.5) * torch.tensor([1.0, 2.0]))
    # pairs (i, i + n/2): a quarter turn of the first pair, 0.01 rad of the second at position 1
    v = torch.tensor([[1.0, 2.0, 3.0, 4.0]])
    r = po.rotate_half_pairs(v, torch.tensor([1]), 100.0 ** 2)
    c0, s0, c1, s1 = [float(f(torch.tensor(a, dtype=torch.float64))) for a in (1.0, 0.01) for f in (torch.cos, torch.sin)]
    assert torch.allclose(r, torch.tensor([[c0 - 3 * s0, 2 * c1 - 4 * s1, 3 * c0 + s0, 4 * c1 + 2 * s1]]), atol=1e-6)
    m = po.window_mask(5, 2)
    assert m.sum(-1).tolist() == [1, 2, 2, 2, 2] and m[4].tolist() == [False, False, False, True, True]
    # one channel: state 0.5 s + 0.5 v
    o, st = po.hgrn2_recurrence(torch.ones(2, 1, 1), torch.full((2, 1, 1), 0.5), torch.tensor([[[2.0]], [[4.0]]]))
    assert o.view(-1).tolist() == [1.0, 2.5] and st.item() == 2.5
    g = po.clamped_glu(torch.tensor([5.0, -9.0]), torch.tensor([-7.0, 0.5]), 2.0)
    s = torch.sigmoid(torch.tensor([1.702 * 2.0, 1.702 * -9.0]))
    assert torch.allclose(g, torch.tensor([2.0, -9.0]) * s * torch.tensor([-1.0, 1.5]))
    idx, sc = po.route(torch.eye(3), torch.tensor([[0.0, 3.0, 1.0], [2.0, 1.0, 0.0]]), 1)
    assert idx.view(-1).tolist() == [1, 0, 0] and torch.allclose(sc.view(-1), torch.sigmoid(torch.tensor([2.0, 3.0, 1.0])))


def test_oracle_is_causal_and_windowed():
    """Changing a token changes nothing before it; with attention layers only, nothing past the last window that
    holds it."""
    cfg = pu.config(32, 50, [(pu.latent(2, 8, 4, 8, 12, 5), pu.experts(3, 2, 8)), (pu.latent(2, 8, 4, 8, 12, 4), None)])
    w = pu.weights(cfg, 1)
    a = pu.tokens(cfg, 30)
    b = a.clone()
    b[10] = (b[10] + 1) % 50
    d = (pu.reference(cfg, w, a, torch.float64) - pu.reference(cfg, w, b, torch.float64)).abs().amax(-1)
    assert d[:10].max() == 0 and d[10] > 1e-3 and d[10 + 4 + 3] > 1e-6 and d[10 + 4 + 3 + 1:].max() == 0


def test_model_class_by_config(tmp_path):
    from gpt_fast import gpt_dense_TP, gpt_ladder_TP, gpt_patevik_TP, loader
    cfg = pu.CONFIGS["uneven"]
    pu.save(cfg, {}, tmp_path / "p")
    cls, args = loader.model_class(str(tmp_path / "p"))
    assert cls is gpt_patevik_TP.GPTPatevik and args.n_layer == 4 and args.dim == 96 and torch.float32 in cls.dtypes
    llama = dict(num_hidden_layers=2, vocab_size=64, num_attention_heads=4, hidden_size=64, intermediate_size=128)
    for extra, want in (({}, gpt_dense_TP.GPTDense), ({"ladder_layers": 1}, gpt_ladder_TP.GPTLadder)):
        os.makedirs(tmp_path / want.__name__, exist_ok=True)
        json.dump(dict(llama, **extra), open(tmp_path / want.__name__ / "config.json", "w"))
        cls, _ = loader.model_class(str(tmp_path / want.__name__))
        assert cls is want and torch.float32 not in cls.dtypes
    json.dump(dict(cfg, architecture="Other"), open(tmp_path / "p" / "config.json", "w"))
    with pytest.raises(ValueError, match="unknown architecture"):
        loader.model_class(str(tmp_path / "p"))


def test_bad_configurations_are_refused():
    from gpt_fast import mixers
    with pytest.raises(ValueError, match="unknown mixer"):
        mixers.make_mixer("other", 8, {})
    m = pu.latent(1, 8, 4, 8, 8, 5)["mixer"]
    with pytest.raises(ValueError, match="rot_dim"):
        mixers.make_mixer("latent_attention", 8, dict(m, rot={"base": 1e4, "dims": 2}))
    with pytest.raises(ValueError, match="even"):
        mixers.make_mixer("latent_attention", 8, dict(m, rot_dim=3, rot={"base": 1e4, "dims": 3}))
    with pytest.raises(ValueError, match="unknown feed-forward"):
        mixers.make_mlp(8, {"kind": "other"})
    with pytest.raises(ValueError, match="top"):
        mixers.make_mlp(8, pu.experts(2, 3, 8))


def test_checkpoint_round_trip_and_missing_tensor(tmp_path):
    from gpt_fast import loader
    cfg = pu.CONFIGS["ones"]
    w = pu.weights(cfg, 2)
    pu.save(cfg, w, tmp_path)
    model = loader.load_model(str(tmp_path), torch.bfloat16, "cpu")
    b = model.layers[0].mixer
    assert torch.equal(b.in_proj.weight[:64], w["l0.rg1"]) and torch.equal(b.in_proj.weight[64:64 + 18], w["l0.mix.q"])
    assert torch.equal(b.in_proj.weight[82:82 + 18], w["l0.mix.dkv"]) and b.in_proj.weight[100:].abs().sum() == 0
    assert b.in_proj.weight.shape[0] % 8 == 0
    moe = model.layers[0].mlp.sublayer
    assert torch.equal(moe.w1[0, :16], w["l0.mlp.e0.up"]) and torch.equal(moe.w1[0, 16:], w["l0.mlp.e0.gate"])
    with pytest.raises(TypeError):
        loader.load_model(str(tmp_path), torch.float64, "cpu")
    del w["l1.mix.f.b"]
    pu.save(cfg, w, tmp_path)
    with pytest.raises(KeyError):
        loader.load_model(str(tmp_path), torch.bfloat16, "cpu")


def test_presets_build():
    from gpt_fast import gpt_patevik_TP as pk
    for name in pk.transformer_configs:
        with torch.device("meta"):
            model = pk.GPTPatevik.from_name(name)
        assert len(model.layers) == model.config.n_layer
    kinds = [b.mixer.sublayer.kind for b in model.layers]
    assert kinds[:2] == ["hgrn2", "latent_attention"]


def test_layer_entry_points_check_arguments_without_a_gpu():
    from gpt_fast import _C
    lib = _C.lib
    assert lib.lri_linear_f32(0, None, None, None, 1, 8, 8, None, 0, None) == -1
    assert lib.lri_linear_f32(5, 16, 16, 16, 1, 8, 8, None, 0, None) == -3
    assert lib.lri_moe_route(16, 8, 4, 5, 1, 16, 16, None, None, None) == -3 and b"experts" in lib.lri_last_error()
    assert lib.lri_hgrn2(0, 16, 8, 0, 4, 8, 16, 16, 16, 1e-5, 16, 16, 0, 16, 1, 4, 1, 600, 8, None, 0, None) == -3
    assert lib.lri_hgrn2(0, 16, 8, 0, 4, 8, 16, 16, 16, 1e-5, 16, 16, 0, 16, 1, 4, 1, 4, 4, None, 0, None) == -5
    assert lib.lri_moe_packs(0, 100, 2, 64, 64) == 1 and lib.lri_moe_packs(2, 100, 2, 64, 64) == 0
    assert lib.lri_moe_packs(0, 4, 2, 64, 64) == 0 and lib.lri_moe_packs(0, 100, 2, 64, 60) == 0
    # every distribution of pairs over experts fits: full tiles plus one partial tile per expert
    assert lib.lri_moe_max_tiles(300, 2, 7) == 600 // 128 + 7 and lib.lri_moe_max_tiles(1, 2, 7) == 2
    # a longer prompt's workspace serves a shorter one
    sizes = [lib.lri_hgrn2_workspace_bytes(0, 1, s, 4, 64, 64) for s in range(16, 1200, 8)]
    assert sizes == sorted(sizes)
