"""Model presets shared by the four schedule families.

The reference keeps one `transformer_configs` dict per family file
(gpt_fast/gpt_ladder_TP.py:65-207, gpt_dense_TP.py:63-182, gpt_parallel_TP.py:63-133,
gpt_desync_TP.py:68-249) with mostly equal entries.  Here every architecture is written once
and each family lists which names it offers and which schedule flags it attaches, so that
`family:preset` strings accepted by the reference's benchmark driver resolve to the same shapes.
Two presets are added for shapes the reference does not have (8 KV heads for the 1B and 405B
Ladder-Llama shapes).
"""
from copy import deepcopy

_LLAMA31_SCALING = dict(factor=8.0, low_freq_factor=1.0, high_freq_factor=4.0, original_max_position_embeddings=8192)


def _arch(n_layer, n_head, dim, **kw):
    return dict(n_layer=n_layer, n_head=n_head, dim=dim, **kw)


def _star(n_layer, n_head, dim, inter):
    # StarCoder-style research shapes: MHA, vocab 49152, 2k context
    return _arch(n_layer, n_head, dim, block_size=2048, n_local_heads=n_head, intermediate_size=inter,
                 vocab_size=49152, rope_base=10000)


def _llama3(n_layer, n_head, dim, inter, **kw):
    return _arch(n_layer, n_head, dim, block_size=8192, n_local_heads=8, intermediate_size=inter,
                 vocab_size=128256, rope_base=500000, **kw)


ARCH = {
    "CodeLlama-7b-Python-hf": _arch(32, 32, 4096, block_size=16384, vocab_size=32000, rope_base=1000000),
    "1b": _star(40, 24, 1536, 4096),
    "1.55b": _star(52, 24, 1536, 4096),
    "3b": _star(40, 32, 2304, 9216),
    "3b-36h": _star(40, 36, 2304, 9216),
    "3.9bh": _star(52, 32, 2304, 9216),
    "3.9bw1": _star(40, 32, 3200, 9216),
    "3.9bw2": _star(40, 32, 2560, 11000),
    "7B": _arch(32, 32, 4096),
    "13B": _arch(40, 40, 5120),
    "30B": _arch(60, 52, 6656),
    "34B": _arch(48, 64, 8192, vocab_size=32000, n_local_heads=8, intermediate_size=22016, rope_base=1000000),
    "70B": _arch(80, 64, 8192, n_local_heads=8, intermediate_size=28672),
    "Mistral-7B": _arch(32, 32, 4096, n_local_heads=8, intermediate_size=14336, vocab_size=32000),
    "stories15M": _arch(6, 6, 288),
    "stories110M": _arch(12, 12, 768),
    "llama-3.2-1b": _arch(16, 32, 2048, intermediate_size=8192, vocab_size=128256),
    "llama-3.2-3b": _arch(28, 24, 3072, intermediate_size=8192, vocab_size=128256),
    "llama-3-8b": _llama3(32, 32, 4096, 14336),
    "llama-3-8b-4layers": _llama3(4, 32, 4096, 14336),
    "llama-3-70b": _llama3(80, 64, 8192, 28672),
    "llama-3.1-405b": _arch(126, 128, 16384, block_size=131072, n_local_heads=16, intermediate_size=53248,
                            vocab_size=128256, rope_base=500000, rope_scaling=_LLAMA31_SCALING),
    "bloom-176b": _arch(70, 112, 14336, block_size=8192, n_local_heads=112, intermediate_size=50176,
                        vocab_size=250880, rope_base=500000),
    # shapes of the headline benchmark that the reference's presets do not cover
    "ladder-llama-1b": _arch(16, 32, 2048, block_size=2048, n_local_heads=8, intermediate_size=8192,
                             vocab_size=128256, rope_base=500000),
    "ladder-llama-405b-kv8": _arch(126, 128, 16384, block_size=131072, n_local_heads=8, intermediate_size=53248,
                                   vocab_size=128256, rope_base=500000, rope_scaling=_LLAMA31_SCALING),
}



def _layer_list(n_layer, width, heads, dim, vdim, kv_rank, rot_dim, window, experts, top, ff, vocab, rope_base=500000.0):
    """Alternating HGRN2 and latent-attention layers of one size, each with a mixture of experts."""
    mlp = dict(kind="moe", expert=dict(ff=ff, limit=7.0), router=dict(experts=experts, top=top))
    recurrent = dict(type="hgrn2", mixer=dict(heads=heads, dim=dim, vdim=vdim), mlp=mlp)
    latent = dict(type="latent_attention", mlp=mlp,
                  mixer=dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, rot_dim=rot_dim, mask=dict(size=window),
                             rot=dict(base=rope_base, dims=rot_dim), scale=(dim + rot_dim) ** -0.5))
    return dict(vocab_size=vocab, dim=width, layers=[deepcopy(latent if i % 2 else recurrent) for i in range(n_layer)])


# Layer-list designs.  The active parameters of a layer's feed-forward are those of the Llama shape of the same name.
LAYER_LISTS = {
    "patevik-tiny": _layer_list(4, 192, 3, 32, 64, 48, 32, 40, 6, 2, 96, 512),
    "patevik-1b": _layer_list(16, 2048, 32, 64, 64, 256, 32, 1024, 8, 2, 4096, 128256),
    "patevik-8b": _layer_list(32, 4096, 32, 128, 128, 512, 64, 4096, 8, 2, 7168, 128256),
}



def _stream_list(n_layer, width, streams, left, right, gla, ff, vocab, every=3):
    """Layers with two mixers side by side, every `every`-th one gated linear attention; a dense unit behind each.
    left (heads, kv_heads, dim, chunk), right (heads, kv_heads, dim, rank), gla (heads, dim, vdim, rank)."""
    mlp = dict(kind="dense", ff=ff, limit=7.0)
    lh, lk, ld, chunk = left
    rh, rk, rd, rank = right
    gh, gd, gv, grank = gla
    side_by_side = dict(type="parallel", mlp=mlp, mixer=dict(
        left_scale=1.0, right_scale=1.0,
        left=dict(heads=lh, kv_heads=lk, dim=ld, vdim=ld, scale=ld ** -0.5, mask=dict(size=chunk), rot=dict(base=500000.0, dims=ld // 2)),
        right=dict(heads=rh, kv_heads=rk, dim=rd, vdim=rd, conv=4, decay_rank=rank, gate_rank=rank)))
    linear = dict(type="gla", mlp=mlp, mixer=dict(heads=gh, dim=gd, vdim=gv, tau=16.0, decay_rank=grank))
    return dict(vocab_size=vocab, dim=width, streams=streams, embed_scale=1.0,
                layers=[deepcopy(linear if i % every == every - 1 else side_by_side) for i in range(n_layer)])


# Residual streams with dense feed-forwards: width, depth, vocabulary and feed-forward of the Llama shape of the same name.
STREAM_LISTS = {
    "migosun-tiny": _stream_list(4, 192, 3, (6, 2, 32, 48), (4, 2, 32, 16), (3, 32, 64, 8), 320, 512),
    "migosun-1b": _stream_list(16, 2048, 4, (32, 8, 64, 4096), (16, 16, 64, 64), (16, 64, 128, 16), 8192, 128256),
    "migosun-8b": _stream_list(32, 4096, 4, (32, 8, 128, 8192), (16, 16, 128, 128), (16, 128, 256, 16), 14336, 128256),
}

_COMMON = ["CodeLlama-7b-Python-hf", "1b", "3b", "7B", "13B", "30B", "34B", "70B", "Mistral-7B", "stories15M",
           "stories110M", "llama-3.2-1b", "llama-3.2-3b", "llama-3-8b", "llama-3-70b", "llama-3.1-405b",
           "ladder-llama-1b", "ladder-llama-405b-kv8"]
_WIDE = ["3.9bh", "3.9bw1", "3.9bw2"]


def _no_reduce(n_layer):
    return [{"attention": False, "mlp": False} for _ in range(n_layer)]


def _every_other_mlp(n_layer):
    return [{"attention": False, "mlp": False}, {"attention": False, "mlp": True}] * (n_layer // 2)


def family_presets(family):
    """Returns {preset name: ModelArgs kwargs} for 'ladder', 'dense', 'parallel', 'desync', 'patevik' or 'migosun'."""
    if family == "migosun":
        return deepcopy(STREAM_LISTS)
    if family == "patevik":
        return deepcopy(LAYER_LISTS)
    out = {}

    def add(name, arch=None, **extra):
        cfg = deepcopy(ARCH[arch or name])
        cfg.update(extra)
        out[name] = cfg

    names = list(_COMMON)
    if family in ("ladder", "dense"):
        names += _WIDE
    if family == "ladder":
        names += ["1.55b", "bloom-176b"]
    if family == "dense":
        names += ["llama-3-8b-4layers"]
    for n in names:
        add(n)
    add("70B-semi-compiled", "70B", semi_compiled_model=True)
    if family == "ladder":
        add("llama-3-8b-semi-compiled", "llama-3-8b", semi_compiled_model=True)
        add("llama-3-70b-semi-compiled", "llama-3-70b", semi_compiled_model=True)
    if family == "desync":
        # In the reference's desync table the plain "1b" entry carries the no-reduce pattern and
        # "1b-upper-bound" the default one; "3b" uses 36 heads.  Kept as they are.
        add("1b", "1b", reduce_pattern=_no_reduce(40), force_disable_last_all_reduce=True)
        add("1b-upper-bound", "1b")
        add("3b", "3b-36h")
        add("3b-upper-bound", "3b-36h", reduce_pattern=_no_reduce(40), force_disable_last_all_reduce=True)
        add("70B-infinite", "70B", reduce_pattern=_no_reduce(80))
        add("70B-infinite-semi-compiled", "70B", semi_compiled_model=True, reduce_pattern=_no_reduce(80))
        for base, layers in (("llama-3-8b", 32), ("llama-3-70b", 80)):
            add(base + "-4x", base, reduce_pattern=_every_other_mlp(layers))
            add(base + "-upper-bound", base, reduce_pattern=_no_reduce(layers), force_disable_last_all_reduce=True)
        add("llama-3-8b-infinite", "llama-3-8b", reduce_pattern=_no_reduce(32))
        add("llama-3.1-405b-upper-bound", "llama-3.1-405b", reduce_pattern=_no_reduce(126),
            force_disable_last_all_reduce=True)
        add("ladder-llama-405b-kv8-upper-bound", "ladder-llama-405b-kv8", reduce_pattern=_no_reduce(126),
            force_disable_last_all_reduce=True)
    return out
