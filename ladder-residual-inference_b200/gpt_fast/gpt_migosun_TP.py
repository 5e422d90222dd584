"""Migosun: a decoder of heterogeneous layers (chunked attention and a gated delta rule side by side, or gated linear
attention), each followed by a dense gated unit or nothing, over a residual of several streams; input and output embeddings
are one table.  No counterpart in the reference project; it runs through the same model shell, engine heads, caches set-up
and decode loop as the other families."""
from copy import deepcopy
from dataclasses import dataclass, field
from typing import Dict, List, Tuple

import torch
import torch.nn as nn

from .engine_layers import LayerEngine
from .mixers import StreamBranch, make_mixer, make_mlp
from .model_base import BlockBase, TPModelBase, args_from_name
from .presets import family_presets
from .tp import maybe_init_dist

maybe_init_dist()

transformer_configs = family_presets("migosun")


@dataclass
class ModelArgs:
    vocab_size: int
    dim: int
    streams: int
    # one entry per layer: {"type", "mixer": {...}, "mlp": {...} or None}
    layers: List[dict] = field(default_factory=list)
    embed_scale: float = 1.0
    norm_eps: float = 1e-5
    block_size: int = 131072
    semi_compiled_model: bool = False

    @property
    def n_layer(self) -> int:
        return len(self.layers)

    @classmethod
    def from_name(cls, name: str):
        return args_from_name(cls, transformer_configs, name)

    @classmethod
    def from_config(cls, c: dict, shapes: Dict[str, Tuple[int, ...]]):
        """From a checkpoint's config.json and the shapes of its tensors, which give the ranks of low-rank projections."""
        layers = deepcopy(c["layers"])
        for i, layer in enumerate(layers):
            mixer, prefix = layer["mixer"], f"l{i}.mix."
            if layer["type"] == "parallel":
                mixer, prefix = mixer["right"], prefix + "right."
                mixer["gate_rank"] = shapes[prefix + "g1"][0]
            mixer["decay_rank"] = shapes[prefix + "a1"][0]
        return cls(vocab_size=c["vocab"], dim=c["width"], streams=c["streams"], layers=layers, embed_scale=c["embedding"]["scale"],
                   norm_eps=c["norm"]["eps"])


class MigosunBlock(BlockBase):
    def __init__(self, config: ModelArgs, layer: dict) -> None:
        super().__init__()
        self.semi_compiled_model = config.semi_compiled_model
        self.mixer = StreamBranch(config.dim, config.streams, make_mixer(layer["type"], config.dim, layer["mixer"]))
        mlp = layer.get("mlp")
        self.mlp = StreamBranch(config.dim, config.streams, make_mlp(config.dim, mlp)) if mlp is not None else None


class GPTMigosun(TPModelBase):
    family = "migosun"
    engine_class = LayerEngine
    dtypes = (torch.bfloat16, torch.float16, torch.float32)

    def __init__(self, config: ModelArgs) -> None:
        super().__init__(config, (MigosunBlock(config, layer) for layer in config.layers))
        self._tie()

    def _tie(self):
        self.output.weight = self.tok_embeddings.weight

    def _apply(self, fn, recurse=True):
        # moving or materialising a module replaces its parameters one by one
        super()._apply(fn, recurse)
        self._tie()
        return self

    @classmethod
    def from_name(cls, name: str):
        return cls(ModelArgs.from_name(name))

    def _setup_layer_caches(self, max_batch_size, max_seq_length, dtype, device):
        for block in self.layers:
            block.mixer.sublayer.setup_cache(max_batch_size, max_seq_length, dtype, device)

    def recurrent_state(self):
        return [t for b in self.layers for t in b.mixer.sublayer.recurrent_state()]

    @torch.no_grad()
    def init_random_(self, std: float = 0.02) -> None:
        """Random weights for measurements: matrices N(0, std), norms 1, streams equal, decays spread, padding zero."""
        for name, p in self.named_parameters():
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("pre_norm", "q_norm", "k_norm", "norm") or name == "norm.weight":
                p.fill_(1.0)
            elif leaf in ("w_in", "w_out"):
                p.fill_(1.0 / p.numel() if leaf == "w_in" else 1.0)
            elif leaf == "w_mix":
                p.copy_(torch.eye(p.shape[0], device=p.device))
            elif leaf in ("sink", "a2_bias"):
                p.zero_()
            elif leaf == "a_log":
                p.copy_(torch.linspace(-4.0, 0.0, p.numel(), device=p.device))
            elif leaf == "dt_bias":
                p.copy_(torch.linspace(-3.0, 1.0, p.numel(), device=p.device))
            elif leaf.startswith("conv_"):
                nn.init.normal_(p, mean=0.0, std=0.5)
            else:
                nn.init.normal_(p, mean=0.0, std=std)
