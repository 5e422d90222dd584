"""Small random Migosun models for the tests: configurations, checkpoint-named weights, and model building."""
import torch

from oracle import migosun_oracle as mo
from patevik_util import feed, row_err, save, tokens  # noqa: F401  (the same for every layer-list design)


def side_by_side(left, right, scales=(0.9, 1.2)):
    """left (heads, kv_heads, dim, vdim, chunk, rot_dims, base, scale), right (heads, kv_heads, dim, vdim, taps, ranks)."""
    H, G, d, dv, chunk, rot, base, scale = left
    h, g, c, e, taps, ranks = right
    return {"type": "parallel", "ranks": ranks,
            "mixer": {"left_scale": scales[0], "right_scale": scales[1],
                      "left": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "mask": {"size": chunk}, "scale": scale,
                               "rot": {"base": base, "dims": rot}},
                      "right": {"heads": h, "kv_heads": g, "dim": c, "vdim": e, "conv": taps}}}


def linear(heads, dim, vdim, tau, rank):
    return {"type": "gla", "ranks": rank, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def dense(ff, limit=1.2):
    return {"kind": "dense", "ff": ff, "limit": limit}


def config(width, vocab, streams, layers, eps=1e-5, scale=0.7):
    """-> (config, ranks of the layers' low-rank projections, which a checkpoint holds as shapes only)"""
    cfg = {"architecture": "Migosun", "width": width, "vocab": vocab, "streams": streams, "norm": {"eps": eps},
           "embedding": {"scale": scale},
           "layers": [{"type": la["type"], "mixer": la["mixer"], "mlp": mlp} for la, mlp in layers]}
    return cfg, [la["ranks"] for la, _ in layers]


CONFIGS = {
    # every layer its own sizes, none that the 16-byte kernels take everywhere
    "uneven": config(92, 101, 3, [(side_by_side((6, 2, 20, 12, 17, 6, 500.0, 0.3), (4, 2, 12, 20, 4, (5, 9))), dense(44)),
                                  (linear(3, 14, 10, 7.0, 6), None),
                                  (side_by_side((3, 3, 10, 22, 31, 10, 1e4, 0.25), (6, 3, 9, 7, 2, (3, 4)), (1.0, 0.5)), dense(36, 0.6)),
                                  (linear(2, 40, 36, 16.0, 12), dense(50))]),
    # sizes of the tensor-core and cluster forms, chunk edges inside tiles, wide groups
    "tiles": config(192, 320, 4, [(side_by_side((8, 2, 64, 96, 50, 32, 1e6, 0.2), (4, 2, 64, 64, 3, (16, 24))), dense(160)),
                                  (side_by_side((4, 4, 128, 64, 130, 128, 1e4, 0.11), (2, 1, 128, 128, 4, (8, 8))), dense(200, 2.0)),
                                  (linear(3, 64, 128, 4.0, 16), dense(160))]),
    # degenerate sizes: one stream, one head, a chunk of one, a convolution of one tap, unit scales
    "ones": config(64, 72, 1, [(side_by_side((1, 1, 16, 8, 1, 2, 1e4, 1.0), (1, 1, 8, 16, 1, (1, 1)), (1.0, 1.0)), dense(16)),
                               (side_by_side((2, 1, 8, 8, 2, 8, 100.0, 0.5), (2, 2, 4, 4, 2, (8, 2)), (2.0, -1.0)), None),
                               (linear(1, 8, 8, 1.0, 1), dense(8))], eps=1e-3, scale=1.0),
    # a chunk longer than any prompt, linear layers first, many streams, vocabulary above the width
    "long_chunk": config(128, 640, 6, [(linear(4, 32, 32, 16.0, 16), dense(96)),
                                       (side_by_side((8, 2, 32, 32, 4096, 16, 1e4, 0.2), (4, 4, 32, 48, 4, (12, 12))), dense(96))]),
}


def weights(case, seed=0, storage=torch.bfloat16):
    """Checkpoint tensors, rounded to the storage type; matrices keep the scale of their input."""
    cfg, ranks = case
    g = torch.Generator().manual_seed(seed)
    d, w, s = cfg["width"], {}, cfg["streams"]

    def mat(name, n, k, gain=1.0):
        w[name] = (torch.randn(n, k, generator=g) * gain * k ** -0.5).to(storage)

    def vec(name, n, mean, std):
        w[name] = (torch.randn(n, generator=g) * std + mean).to(storage)

    w["embed"] = torch.randn(cfg["vocab"], d, generator=g).to(storage)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for q in (1, 2) if layer["mlp"] else (1,):
            vec(f"{p}norm{q}", d, 1.0, 0.2)
            vec(f"{p}hc{q}.in", s, 1.0 / s, 0.2)
            vec(f"{p}hc{q}.out", s, 0.8, 0.3)
            w[f"{p}hc{q}.mix"] = (torch.eye(s) + torch.randn(s, s, generator=g) * 0.15).to(storage)
        if layer["type"] == "parallel":
            a, b, x = m["left"], m["right"], p + "mix.left."
            for t, n, gain in (("q", a["heads"] * a["dim"], 1.5), ("k", a["kv_heads"] * a["dim"], 1.5), ("v", a["kv_heads"] * a["vdim"], 1.0)):
                mat(x + t, n, d, gain)
            vec(x + "q.norm", a["heads"] * a["dim"], 1.0, 0.3)
            vec(x + "k.norm", a["kv_heads"] * a["dim"], 1.0, 0.3)
            vec(x + "sink", a["heads"], 1.5, 1.0)
            mat(x + "o", d, a["heads"] * a["vdim"])
            x, H, C, E, qk = p + "mix.right.", b["heads"], b["dim"], b["vdim"], b["kv_heads"] * b["dim"]
            for t, n in (("q", qk), ("k", qk), ("v", H * E)):
                mat(x + t, n, d)
                w[x + t + ".conv"] = (torch.randn(n, b["conv"], generator=g) * b["conv"] ** -0.5).to(storage)
            mat(x + "b", H, d, 1.5)
            vec(x + "A_log", H, -1.5, 1.0)
            mat(x + "a1", ranks[i][0], d)
            mat(x + "a2", H * C, ranks[i][0])
            vec(x + "dt_bias", H * C, -1.0, 1.0)
            mat(x + "g1", ranks[i][1], d)
            mat(x + "g2", H * E, ranks[i][1], 1.5)
            vec(x + "norm", E, 1.0, 0.2)
            mat(x + "o", d, H * E)
        else:
            x, H, C, E = p + "mix.", m["heads"], m["dim"], m["vdim"]
            for t, n in (("q", H * C), ("k", H * C), ("v", H * E), ("g", H * E)):
                mat(x + t, n, d)
            mat(x + "a1", ranks[i], d)
            mat(x + "a2", H * C, ranks[i], 2.0)
            vec(x + "a2.b", H * C, 1.0, 1.0)
            vec(x + "norm", E, 1.0, 0.2)
            mat(x + "o", d, H * E)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            mat(p + "mlp.gate", ff, d, 1.5)
            mat(p + "mlp.up", ff, d, 1.5)
            mat(p + "mlp.down", d, ff)
    vec("final.norm", d, 1.0, 0.2)
    return w


def build(cfg, w, dtype, device, batch, max_seq):
    import torch.distributed as dist
    from gpt_fast import gpt_migosun_TP as mg
    from gpt_fast import loader
    with torch.device("meta"):
        model = mg.GPTMigosun(mg.ModelArgs.from_config(cfg, {k: tuple(v.shape) for k, v in w.items()}))
    model = model.to(dtype=dtype).to_empty(device=device).eval()
    loader._copy_parameters(model, loader.migosun_to_local(w, model, dist.get_rank(), dist.get_world_size()))
    model.setup_caches(max_batch_size=batch, max_seq_length=max_seq)
    return model


def reference(cfg, w, toks, dtype=torch.float32):
    with torch.no_grad():
        return mo.forward(cfg, w, toks, dtype)
