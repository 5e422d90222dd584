"""Patevik: a decoder of heterogeneous layers (latent attention with a sliding window, HGRN2 recurrence), each followed
by a mixture of experts, every sublayer in a gated residual branch with a norm before and after.  No counterpart in the
reference project; it runs through the same model shell, engine heads, caches set-up and decode loop as the other
families."""
from dataclasses import dataclass, field
from typing import List

import torch
import torch.nn as nn

from .engine_layers import LayerEngine
from .mixers import GatedResidual, make_mixer, make_mlp
from .model_base import BlockBase, TPModelBase, args_from_name
from .presets import family_presets
from .tp import maybe_init_dist

maybe_init_dist()

transformer_configs = family_presets("patevik")


@dataclass
class ModelArgs:
    vocab_size: int
    dim: int
    # one entry per layer: {"type", "mixer": {...}, "mlp": {...} or None}
    layers: List[dict] = field(default_factory=list)
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
    def from_config(cls, c: dict):
        """From a checkpoint's config.json."""
        return cls(vocab_size=c["vocab"], dim=c["width"], layers=c["layers"], norm_eps=c["norm"]["eps"])


class PatevikBlock(BlockBase):
    def __init__(self, config: ModelArgs, layer: dict) -> None:
        super().__init__()
        self.semi_compiled_model = config.semi_compiled_model
        self.mixer = GatedResidual(config.dim, make_mixer(layer["type"], config.dim, layer["mixer"]))
        mlp = layer.get("mlp")
        self.mlp = GatedResidual(config.dim, make_mlp(config.dim, mlp)) if mlp is not None else None


class GPTPatevik(TPModelBase):
    family = "patevik"
    engine_class = LayerEngine
    dtypes = (torch.bfloat16, torch.float16, torch.float32)

    def __init__(self, config: ModelArgs) -> None:
        super().__init__(config, (PatevikBlock(config, layer) for layer in config.layers))

    @classmethod
    def from_name(cls, name: str):
        return cls(ModelArgs.from_name(name))

    def _setup_layer_caches(self, max_batch_size, max_seq_length, dtype, device):
        for block in self.layers:
            block.mixer.sublayer.setup_cache(max_batch_size, max_seq_length, dtype, device)

    def recurrent_state(self):
        return [b.mixer.sublayer.kv_cache.state for b in self.layers if b.mixer.sublayer.kind == "hgrn2"]

    @torch.no_grad()
    def init_random_(self, std: float = 0.02) -> None:
        """Random weights for measurements: matrices N(0, std), norms 1, biases 0, forget-gate bounds spread over (0, 1),
        unused rows of the fused projections zero."""
        for name, p in self.named_parameters():
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("pre_norm", "post_norm", "latent_norm", "norm") or name == "norm.weight":
                p.fill_(1.0)
            elif leaf in ("gate_bias", "f_bias"):
                p.zero_()
            elif leaf == "lower":
                p.copy_(torch.linspace(0.0, 0.99, p.numel(), device=p.device))
            else:
                nn.init.normal_(p, mean=0.0, std=std)
        for block in self.layers:
            for branch in (block.mixer, block.mlp):
                if branch is not None:
                    branch.in_proj.weight[branch.width + branch.sublayer.in_rows:].zero_()
