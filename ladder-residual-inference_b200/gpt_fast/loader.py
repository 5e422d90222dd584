"""Checkpoints -> the fused, sharded parameter layout of this package: Hugging Face Llama / LlamaLadder, Patevik and Migosun.
`load_model(path)` picks the model class from the folder's config.json.

The reference has no loader (every rank draws its own random shard, benchmark.py:242-243); the only
conversion it carries is the load hook that fuses separate wq / wk / wv into wqkv
(gpt_fast/utils.py:178-185, kept in this package's Attention).  Real checkpoints of the Ladder
models use the Hugging Face Llama names (reference hf_modeling_utils/modeling_llama_ladder.py:
self_attn.{q,k,v,o}_proj at 281-284, mlp.{gate,up,down}_proj at 235-237); this module maps them onto
the per-rank layout that the kernels read:

    wqkv  [(nh + 2 nkv) hd / t, d]  rows [q heads of the rank | k heads | v heads]
    wo    [d, nh hd / t]            columns of the rank's heads
    w1    [2 I / t, d]              rows [up slice | gate slice]
    w2    [d, I / t]                columns of the slice
    tok_embeddings, output, all norm weights: replicated

Rotary layout: Hugging Face rotates the pairs (i, i + hd/2) of a head ("rotate half"), gpt_fast the
adjacent pairs (2i, 2i + 1) (gpt_fast/utils.py:120-132).  The rows of q_proj and k_proj are
therefore re-ordered inside every head, new row 2i + j = old row j hd/2 + i; scores q.k are
unchanged by a permutation applied to both, and v / o_proj are untouched.
"""
import glob
import json
import os
import struct
from typing import Dict, List, Optional, Tuple

import torch
import torch.distributed as dist
from torch import Tensor


def _interleave_rotary_rows(w: Tensor, n_heads: int, head_dim: int) -> Tensor:
    """[n_heads * head_dim, d] in rotate-half order -> adjacent-pair order."""
    d = w.shape[1]
    return w.view(n_heads, 2, head_dim // 2, d).transpose(1, 2).reshape(n_heads * head_dim, d)


def _rows(w: Tensor, rank: int, world: int) -> Tensor:
    n = w.shape[0] // world
    return w[rank * n:(rank + 1) * n]


def _cols(w: Tensor, rank: int, world: int) -> Tensor:
    n = w.shape[1] // world
    return w[:, rank * n:(rank + 1) * n]


def hf_to_local(hf: Dict[str, Tensor], config, rank: int, world: int, family: str = "ladder") -> Dict[str, Tensor]:
    """State dict of a Hugging Face Llama-style model -> state dict of rank `rank` of `world` for the
    ladder / dense / desync module tree of this package (they share it).  Tensors keep their dtype;
    slices are views where possible."""
    if family == "parallel":
        raise ValueError("the parallel attention/MLP block has one norm per layer; Llama checkpoints do not map onto it")
    nh, nkv, d = config.n_head, config.n_local_heads, config.dim
    hd = d // nh
    inter = config.intermediate_size
    for name, v in (("n_head", nh), ("n_local_heads", nkv), ("intermediate_size", inter), ("dim", d)):
        if v % world:
            raise ValueError(f"{name}={v} is not divisible by the tensor-parallel degree {world}")
    out = {"tok_embeddings.weight": hf["model.embed_tokens.weight"], "norm.weight": hf["model.norm.weight"],
           # tied embeddings: the output projection is the embedding table
           "output.weight": hf.get("lm_head.weight", hf["model.embed_tokens.weight"])}
    for i in range(config.n_layer):
        src = f"model.layers.{i}."
        dst = f"layers.{i}."
        q = _interleave_rotary_rows(hf[src + "self_attn.q_proj.weight"], nh, hd)
        k = _interleave_rotary_rows(hf[src + "self_attn.k_proj.weight"], nkv, hd)
        v = hf[src + "self_attn.v_proj.weight"]
        if tuple(q.shape) != (nh * hd, d) or tuple(k.shape) != (nkv * hd, d) or tuple(v.shape) != (nkv * hd, d):
            raise ValueError(f"layer {i}: projection shapes do not match the preset")
        out[dst + "attention.wqkv.weight"] = torch.cat([_rows(q, rank, world), _rows(k, rank, world), _rows(v, rank, world)])
        out[dst + "attention.wo.weight"] = _cols(hf[src + "self_attn.o_proj.weight"], rank, world)
        out[dst + "feed_forward.w1.weight"] = torch.cat([_rows(hf[src + "mlp.up_proj.weight"], rank, world),
                                                         _rows(hf[src + "mlp.gate_proj.weight"], rank, world)])
        out[dst + "feed_forward.w2.weight"] = _cols(hf[src + "mlp.down_proj.weight"], rank, world)
        out[dst + "attention_norm.weight"] = hf[src + "input_layernorm.weight"]
        out[dst + "ffn_norm.weight"] = hf[src + "post_attention_layernorm.weight"]
    return out


def _fuse_branch(get, name: str, branch, parts, rank: int, world: int) -> Dict[str, Tensor]:
    """Parameters of one gated residual branch; `parts` lists (tensor, "rows" or "all") of the sublayer's input rows."""
    rows = [get(f"{name}.gate")] + [_rows(t, rank, world) if how == "rows" else t for t, how in parts]
    total = branch.in_proj.weight.shape[0]
    have = sum(r.shape[0] for r in rows)
    if have < total:
        rows.append(torch.zeros(total - have, rows[0].shape[1], dtype=rows[0].dtype))
    return {"in_proj.weight": torch.cat(rows), "gate_bias": get(f"{name}.gate_bias"), "pre_norm": get(f"{name}.pre"),
            "post_norm": get(f"{name}.post")}


def patevik_to_local(w: Dict[str, Tensor], model, rank: int, world: int) -> Dict[str, Tensor]:
    """Patevik checkpoint tensors -> state dict of rank `rank` of `world` for GPTPatevik's module tree:

        in_proj   rows [gate of the branch | sublayer's input rows of the rank | zero rows]
        expand    rows [W_uk of the rank's heads | W_uv of the rank's heads]
        w1, w2    stacked experts, rows [up | gate] and columns of the rank's slice of the expert width
    """
    out = {"tok_embeddings.weight": w["embed"], "norm.weight": w["final.norm"], "output.weight": w["head"]}
    for i, block in enumerate(model.layers):
        p = f"l{i}."
        names = {"mixer.gate": "rg1", "mixer.gate_bias": "rg1.b", "mixer.pre": "norm1", "mixer.post": "norm1b",
                 "mlp.gate": "rg2", "mlp.gate_bias": "rg2.b", "mlp.pre": "norm2", "mlp.post": "norm2b"}

        def get(k):
            return w[p + names[k]]

        mixer = block.mixer.sublayer
        parts = [(w[f"{p}mix.{t}"], how) for t, how in mixer.tensors().items()]
        for k, v in _fuse_branch(get, "mixer", block.mixer, parts, rank, world).items():
            out[f"layers.{i}.mixer.{k}"] = v
        dst = f"layers.{i}.mixer.sublayer."
        out[dst + "wo.weight"] = _cols(w[p + "mix.o"], rank, world)
        if mixer.kind == "latent_attention":
            out[dst + "latent_norm"] = w[p + "mix.dkv.norm"]
            out[dst + "expand.weight"] = torch.cat([_rows(w[p + "mix.uk"], rank, world), _rows(w[p + "mix.uv"], rank, world)])
        else:
            out[dst + "f_bias"] = _rows(w[p + "mix.f.b"], rank, world)
            out[dst + "lower"] = _rows(w[p + "mix.lower"], rank, world)
            out[dst + "norm"] = w[p + "mix.norm"]
        if block.mlp is None:
            continue
        moe = block.mlp.sublayer
        for k, v in _fuse_branch(get, "mlp", block.mlp, [(w[p + "mlp.router"], "all")], rank, world).items():
            out[f"layers.{i}.mlp.{k}"] = v
        dst = f"layers.{i}.mlp.sublayer."
        experts = [f"{p}mlp.e{e}." for e in range(moe.experts)]
        out[dst + "w1"] = torch.stack([torch.cat([_rows(w[e + "up"], rank, world), _rows(w[e + "gate"], rank, world)])
                                       for e in experts])
        out[dst + "w2"] = torch.stack([_cols(w[e + "down"], rank, world) for e in experts])
    return out


def _pad_to(w: Tensor, dim: int, n: int) -> Tensor:
    """w with zeros behind it along `dim`, n in all."""
    if w.shape[dim] == n:
        return w
    shape = list(w.shape)
    shape[dim] = n - w.shape[dim]
    return torch.cat([w, torch.zeros(shape, dtype=w.dtype)], dim)


def migosun_to_local(w: Dict[str, Tensor], model, rank: int, world: int) -> Dict[str, Tensor]:
    """Migosun checkpoint tensors -> state dict of rank `rank` of `world` for GPTMigosun's module tree:

        in_proj   the mixer's input rows of the rank, low-rank parts padded with zero rows, zero rows at the end
        a2, g2    rows of the rank's heads, columns padded like the rows they multiply
        wo        columns of the rank's heads; side by side: [left o | right o]
        w1        rows [up | gate] of the rank's slice of the feed-forward width
    """
    out = {"tok_embeddings.weight": w["embed"], "norm.weight": w["final.norm"]}
    for i, block in enumerate(model.layers):
        p = f"l{i}."

        def rows(name):
            return _rows(w[name], rank, world)

        for branch, mine, norm, hc in ((block.mixer, "mixer", "norm1", "hc1"), (block.mlp, "mlp", "norm2", "hc2")):
            if branch is not None:
                dst = f"layers.{i}.{mine}."
                out[dst + "pre_norm"] = w[p + norm]
                for t in ("in", "mix", "out"):
                    out[f"{dst}w_{t}"] = w[f"{p}{hc}.{t}"]
        mixer, src, dst = block.mixer.sublayer, p + "mix.", f"layers.{i}.mixer."
        parts = [_pad_to(rows(src + r.name) if r.split == "rows" else w[src + r.name], 0, r.padded) for r in mixer.parts()]
        out[dst + "in_proj.weight"] = _pad_to(torch.cat(parts), 0, block.mixer.in_proj.weight.shape[0])
        dst += "sublayer."
        if mixer.kind == "parallel":
            left, right = src + "left.", src + "right."
            out[dst + "wo.weight"] = torch.cat([_cols(w[left + "o"], rank, world), _cols(w[right + "o"], rank, world)], 1)
            out[dst + "left.q_norm"], out[dst + "left.k_norm"] = rows(left + "q.norm"), rows(left + "k.norm")
            out[dst + "left.sink"] = rows(left + "sink")
            for t in ("q", "k", "v"):
                out[f"{dst}right.conv_{t}"] = rows(f"{right}{t}.conv")
            out[dst + "right.a2"] = _pad_to(rows(right + "a2"), 1, mixer.right.a2.shape[1])
            out[dst + "right.g2"] = _pad_to(rows(right + "g2"), 1, mixer.right.g2.shape[1])
            out[dst + "right.a_log"], out[dst + "right.dt_bias"] = rows(right + "A_log"), rows(right + "dt_bias")
            out[dst + "right.norm"] = w[right + "norm"]
        else:
            out[dst + "wo.weight"] = _cols(w[src + "o"], rank, world)
            out[dst + "a2"] = _pad_to(rows(src + "a2"), 1, mixer.a2.shape[1])
            out[dst + "a2_bias"] = rows(src + "a2.b")
            out[dst + "norm"] = w[src + "norm"]
        if block.mlp is not None:
            src, dst = p + "mlp.", f"layers.{i}.mlp.sublayer."
            out[dst + "w1"] = torch.cat([rows(src + "up"), rows(src + "gate")])
            out[dst + "w2"] = _cols(w[src + "down"], rank, world)
    return out


def _safetensors_shapes(path: str) -> Dict[str, Tuple[int, ...]]:
    """Shapes of the tensors in a folder's *.safetensors, from the files' headers."""
    out: Dict[str, Tuple[int, ...]] = {}
    for name in sorted(glob.glob(os.path.join(path, "*.safetensors"))):
        with open(name, "rb") as f:
            header = json.loads(f.read(struct.unpack("<Q", f.read(8))[0]))
        out.update({k: tuple(v["shape"]) for k, v in header.items() if k != "__metadata__"})
    return out


def _read_safetensors(path: str) -> Dict[str, Tensor]:
    from safetensors.torch import load_file
    files = sorted(glob.glob(os.path.join(path, "*.safetensors"))) if os.path.isdir(path) else [path]
    if not files:
        raise FileNotFoundError(f"no *.safetensors under {path}")
    out: Dict[str, Tensor] = {}
    for f in files:
        out.update(load_file(f))
    return out


def _copy_parameters(model, local: Dict[str, Tensor]) -> None:
    params = dict(model.named_parameters())
    missing = sorted(set(params) - set(local))
    if missing:
        raise KeyError(f"checkpoint has no tensor for {missing[:4]}{' ...' if len(missing) > 4 else ''}")
    with torch.no_grad():
        for name, p in params.items():
            src = local[name]
            if tuple(src.shape) != tuple(p.shape):
                raise ValueError(f"{name}: checkpoint shard {tuple(src.shape)} vs parameter {tuple(p.shape)}")
            p.copy_(src.to(device=p.device, dtype=p.dtype))


def _patevik_class(config: dict, path: str):
    from .gpt_patevik_TP import GPTPatevik, ModelArgs
    return GPTPatevik, ModelArgs.from_config(config)


def _migosun_class(config: dict, path: str):
    from .gpt_migosun_TP import GPTMigosun, ModelArgs
    return GPTMigosun, ModelArgs.from_config(config, _safetensors_shapes(path))


# designs with a checkpoint format of their own: state dict of a rank from the checkpoint's tensors
_LAYOUTS = {"patevik": patevik_to_local, "migosun": migosun_to_local}


def _llama_class(path_or_config):
    """Llama checkpoints run the ladder family when the config names ladder layers, the dense family otherwise."""
    from . import gpt_dense_TP, gpt_ladder_TP
    kw = model_args_from_hf_config(path_or_config)
    if "ladder_layers" in kw:
        return gpt_ladder_TP.GPTLadder, gpt_ladder_TP.ModelArgs(**kw)
    return gpt_dense_TP.GPTDense, gpt_dense_TP.ModelArgs(**kw)


def model_class(path: str):
    """(model class, model args) of the checkpoint folder `path`, by its config.json: `architecture` for designs with
    their own format, otherwise the Hugging Face Llama fields."""
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    name = config.get("architecture")
    if name is None:
        return _llama_class(path)
    known = {"Patevik": _patevik_class, "Migosun": _migosun_class}
    if name not in known:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(known)}")
    return known[name](config, path)


def load_model(path: str, dtype=torch.bfloat16, device="cuda", max_batch_size: Optional[int] = None,
               max_seq_length: Optional[int] = None):
    """Model of the checkpoint folder `path` on `device`, in `dtype`, this rank's shard; caches set up when both
    sizes are given."""
    cls, args = model_class(path)
    if dtype not in cls.dtypes:
        raise TypeError(f"{cls.__name__} runs in {[str(d) for d in cls.dtypes]}, not {dtype}")
    with torch.device("meta"):
        model = cls(args)
    model = model.to(dtype=dtype).to_empty(device=device).eval()
    rank, world = dist.get_rank(), dist.get_world_size()
    tensors = _read_safetensors(path)
    if cls.family in _LAYOUTS:
        _copy_parameters(model, _LAYOUTS[cls.family](tensors, model, rank, world))
    else:
        load_hf_state_dict(model, tensors, rank, world)
    if max_batch_size is not None and max_seq_length is not None:
        model.setup_caches(max_batch_size=max_batch_size, max_seq_length=max_seq_length)
    return model


def model_args_from_hf_config(path: str) -> Dict[str, object]:
    """ModelArgs keyword arguments from the config.json of a Hugging Face Llama / LlamaLadder
    checkpoint directory (field names: transformers' LlamaConfig; `ladder_layers` as normalised by
    the reference's hf_modeling_utils/configuration_llama_ladder.py:38-45).  Register the result under
    a preset name in a family's `transformer_configs` and build the model with `from_name`."""
    with open(os.path.join(path, "config.json") if os.path.isdir(path) else path) as f:
        c = json.load(f)
    n_layer = c["num_hidden_layers"]
    kw = dict(block_size=c.get("max_position_embeddings", 2048), vocab_size=c["vocab_size"], n_layer=n_layer,
              n_head=c["num_attention_heads"], n_local_heads=c.get("num_key_value_heads", c["num_attention_heads"]),
              dim=c["hidden_size"], intermediate_size=c["intermediate_size"], rope_base=c.get("rope_theta", 10000.0),
              norm_eps=c.get("rms_norm_eps", 1e-5))
    scaling = c.get("rope_scaling")
    if scaling and scaling.get("rope_type", scaling.get("type")) == "llama3":
        kw["rope_scaling"] = {k: scaling[k] for k in ("factor", "low_freq_factor", "high_freq_factor",
                                                       "original_max_position_embeddings")}
    if "ladder_layers" in c:
        ll = c["ladder_layers"]
        if ll is None:
            ll = []
        elif isinstance(ll, int):
            ll = list(range(n_layer - ll, n_layer))
        kw["ladder_layers"] = [int(i) for i in ll]
    return kw


def load_hf_state_dict(model, hf: Dict[str, Tensor], rank: Optional[int] = None, world: Optional[int] = None) -> None:
    """Copies a Hugging Face Llama-style state dict into `model` (a GPTLadder / GPTDense / GPTDesync
    of this package, already on its device and in its dtype), taking this rank's shard."""
    rank = dist.get_rank() if rank is None else rank
    world = dist.get_world_size() if world is None else world
    local = hf_to_local(hf, model.config, rank, world, model.family)
    _copy_parameters(model, local)


def load_hf_checkpoint(model, path: str, rank: Optional[int] = None, world: Optional[int] = None) -> None:
    """`path`: a directory of *.safetensors shards (or one file) in Hugging Face Llama naming."""
    load_hf_state_dict(model, _read_safetensors(path), rank, world)
