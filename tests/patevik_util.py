"""Small random Patevik models for the tests: configurations, checkpoint-named weights, and model building."""
import json
import os

import torch

from oracle import patevik_oracle as po


def latent(heads, dim, rot_dim, vdim, rank, window, base=10000.0, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def recurrent(heads, dim, vdim):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def experts(n, top, ff, limit=1.5):
    return {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff, "limit": limit}}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Patevik", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "layers": [dict(layer, mlp=mlp) for layer, mlp in layers]}


CONFIGS = {
    # every layer its own sizes, widths that the 16-byte kernels do not take
    "uneven": config(96, 101, [(latent(3, 20, 6, 12, 36, 17, 500.0), experts(5, 2, 40)), (recurrent(2, 12, 20), experts(3, 1, 24)),
                               (recurrent(5, 16, 8), None), (latent(2, 24, 8, 40, 48, 31), experts(7, 3, 20))]),
    # sizes of the tensor-core forms, window edges inside tiles
    "tiles": config(192, 320, [(recurrent(2, 64, 64), experts(6, 2, 72)), (latent(6, 64, 32, 64, 128, 50), experts(6, 2, 72)),
                               (recurrent(3, 48, 80), experts(4, 4, 64, 0.5)), (latent(3, 40, 16, 72, 96, 130, 1e6, 0.2), experts(6, 1, 88))]),
    # degenerate sizes: a window of one, one head, one expert, no feed-forward
    "ones": config(64, 72, [(latent(1, 16, 2, 16, 16, 1), experts(1, 1, 16)), (recurrent(1, 8, 16), None),
                            (latent(1, 8, 4, 8, 8, 2), None)], eps=1e-3),
    # window longer than any prompt, only attention first, vocabulary above the width
    "wide_window": config(128, 640, [(latent(4, 32, 16, 32, 64, 4096), experts(8, 2, 48)), (recurrent(4, 128, 128), experts(8, 2, 48))]),
}


def weights(cfg, seed=0, storage=torch.bfloat16):
    """Checkpoint tensors, rounded to the storage type; matrices keep the scale of their input."""
    g = torch.Generator().manual_seed(seed)
    d, w = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        w[name] = (torch.randn(n, k, generator=g) * gain * k ** -0.5).to(storage)

    def vec(name, n, mean, std):
        w[name] = (torch.randn(n, generator=g) * std + mean).to(storage)

    w["embed"] = torch.randn(cfg["vocab"], d, generator=g).to(storage)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        names = ["norm1", "norm1b"] + (["norm2", "norm2b"] if layer["mlp"] else [])
        for n in names:
            vec(p + n, d, 1.0, 0.2)
        for n in ["rg1"] + (["rg2"] if layer["mlp"] else []):
            mat(p + n, d, d)
            vec(p + n + ".b", d, 0.3, 0.5)
        H = m["heads"]
        mat(p + "mix.o", d, H * m["vdim"])
        if layer["type"] == "hgrn2":
            mat(p + "mix.q", H * m["dim"], d)
            mat(p + "mix.f", H * m["dim"], d)
            mat(p + "mix.v", H * m["vdim"], d)
            vec(p + "mix.f.b", H * m["dim"], 1.0, 1.0)
            w[p + "mix.lower"] = torch.linspace(0, 0.95, H * m["dim"])[torch.randperm(H * m["dim"], generator=g)].to(storage)
            vec(p + "mix.norm", m["vdim"], 1.0, 0.2)
        else:
            mat(p + "mix.q", H * (m["dim"] + m["rot_dim"]), d, 1.5)
            mat(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], d, 1.5)
            vec(p + "mix.dkv.norm", m["kv_rank"], 1.0, 0.2)
            mat(p + "mix.uk", H * m["dim"], m["kv_rank"])
            mat(p + "mix.uv", H * m["vdim"], m["kv_rank"])
        if layer["mlp"]:
            ff = layer["mlp"]["expert"]["ff"]
            mat(p + "mlp.router", layer["mlp"]["router"]["experts"], d, 2.0)
            for e in range(layer["mlp"]["router"]["experts"]):
                mat(p + f"mlp.e{e}.gate", ff, d, 2.0)
                mat(p + f"mlp.e{e}.up", ff, d, 2.0)
                mat(p + f"mlp.e{e}.down", d, ff)
    vec("final.norm", d, 1.0, 0.2)
    mat("head", cfg["vocab"], d)
    return w


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed))


def save(cfg, w, path):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))


def build(cfg, w, dtype, device, batch, max_seq):
    import torch.distributed as dist
    from gpt_fast import gpt_patevik_TP as pk
    from gpt_fast import loader
    with torch.device("meta"):
        model = pk.GPTPatevik(pk.ModelArgs.from_config(cfg))
    model = model.to(dtype=dtype).to_empty(device=device).eval()
    loader._copy_parameters(model, loader.patevik_to_local(w, model, dist.get_rank(), dist.get_world_size()))
    model.setup_caches(max_batch_size=batch, max_seq_length=max_seq)
    return model


def reference(cfg, w, toks, dtype=torch.float32):
    with torch.no_grad():
        return po.forward(cfg, w, toks, dtype)


def feed(model, toks, cuts, start=0, device="cuda"):
    """Logits of every position of [B, n] tokens fed in portions of the given sizes (the last one repeats)."""
    out, at, i = [], 0, 0
    n = toks.shape[1]
    while at < n:
        k = min(cuts[min(i, len(cuts) - 1)], n - at)
        pos = torch.arange(start + at, start + at + k, dtype=torch.int32, device=device)
        with torch.no_grad():
            out.append(model(toks[:, at:at + k].to(device), pos).float().cpu())
        at, i = at + k, i + 1
    return torch.cat(out, dim=1)


def row_err(got, ref):
    """Relative error of every row of logits, mean taken off."""
    a, b = got - got.mean(-1, keepdim=True), ref - ref.mean(-1, keepdim=True)
    return (a - b).norm(dim=-1) / b.norm(dim=-1)
