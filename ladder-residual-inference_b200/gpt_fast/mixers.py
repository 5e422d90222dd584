"""Sublayers of layer-list designs: latent attention, the HGRN2 recurrence and a mixture of experts, with the caches they
keep.  Beside the Llama sublayers of `utils`, with every size and constant a constructor argument.

Modules own parameters and cache buffers in the layout the kernels read; `engine_layers.LayerEngine` runs them.
Tensor parallelism is fixed at construction as everywhere in the package: heads and expert widths are divided by the
world size, projections from the model width are split by rows, projections back to it by columns.

A sublayer's input projections are fused with the projection of the gate that scales its result (see
`GatedResidual`): `in_proj` rows = [gate (width) | sublayer rows | zero rows up to a multiple of 8].
"""
import math
from typing import Dict

import torch
import torch.nn as nn
from torch import Tensor

from .utils import tp_world_size


def _divide(what: str, n: int, by: int) -> int:
    if n % by:
        raise ValueError(f"{what}={n} is not divisible by the tensor-parallel degree {by}")
    return n // by


def rotate_half_table(positions: int, dims: int, base: float, device) -> Tensor:
    """fp32 [positions, dims/2, 2] = (cos, sin) of p * base^(-2i/dims), evaluated in fp64."""
    i = torch.arange(dims // 2, dtype=torch.float64, device=device)
    ang = torch.outer(torch.arange(positions, dtype=torch.float64, device=device), torch.exp(-(2.0 * i / dims) * math.log(base)))
    return torch.stack([torch.cos(ang), torch.sin(ang)], dim=-1).float().contiguous()


class LatentCache(nn.Module):
    """One row [latent | rotated key] per token: [max_batch, max_seq, rank + rot_dim]."""

    def __init__(self, max_batch_size, max_seq_length, rank, rot_dim, dtype):
        super().__init__()
        self.register_buffer("rows", torch.zeros(max_batch_size, max_seq_length, rank + rot_dim, dtype=dtype))


class RecurrentState(nn.Module):
    """fp32 state [max_batch, heads, dim, vdim] that a call at position 0 restarts and any other call continues."""

    def __init__(self, max_batch_size, heads, dim, vdim):
        super().__init__()
        self.register_buffer("state", torch.zeros(max_batch_size, heads, dim, vdim, dtype=torch.float32))


class LatentAttention(nn.Module):
    """Attention over per-token latents with a sliding window.  in_rows = [q: heads of (dim | rot_dim) | latent | key part]."""

    kind = "latent_attention"

    def __init__(self, width: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, window: int, scale: float,
                 rot_base: float):
        super().__init__()
        if rot_dim % 2 or window < 1:
            raise ValueError(f"latent attention: rot_dim={rot_dim} must be even and the window ({window}) at least 1")
        self.heads = _divide("heads", heads, tp_world_size)
        self.dim, self.rot_dim, self.vdim, self.rank = dim, rot_dim, vdim, kv_rank
        self.window, self.scale, self.rot_base = window, scale, rot_base
        self.q_rows = self.heads * (dim + rot_dim)
        self.in_rows = self.q_rows + kv_rank + rot_dim
        self.latent_norm = nn.Parameter(torch.ones(kv_rank))
        # rows [per-head keys | per-head values] of the latent
        self.expand = nn.Linear(kv_rank, self.heads * (dim + vdim), bias=False)
        self.wo = nn.Linear(self.heads * vdim, width, bias=False)
        self.kv_cache = None

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def setup_cache(self, max_batch, max_seq, dtype, device):
        self.kv_cache = LatentCache(max_batch, max_seq, self.rank, self.rot_dim, dtype).to(device)
        self.rope_table = rotate_half_table(max_seq, self.rot_dim, self.rot_base, device)

    def tensors(self) -> Dict[str, str]:
        """Checkpoint names of the input rows, in order, and how each is split over ranks."""
        return {"q": "rows", "dkv": "all"}


class HGRN2(nn.Module):
    """Linear attention with a bounded forget gate.  in_rows = [q | f | v]."""

    kind = "hgrn2"

    def __init__(self, width: int, heads: int, dim: int, vdim: int):
        super().__init__()
        self.heads = _divide("heads", heads, tp_world_size)
        self.dim, self.vdim = dim, vdim
        self.in_rows = self.heads * (2 * dim + vdim)
        self.f_bias = nn.Parameter(torch.zeros(self.heads * dim))
        self.lower = nn.Parameter(torch.zeros(self.heads * dim))
        self.norm = nn.Parameter(torch.ones(vdim))
        self.wo = nn.Linear(self.heads * vdim, width, bias=False)
        self.kv_cache = None

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def setup_cache(self, max_batch, max_seq, dtype, device):
        self.kv_cache = RecurrentState(max_batch, self.heads, self.dim, self.vdim).to(device)

    def tensors(self) -> Dict[str, str]:
        return {"q": "rows", "f": "rows", "v": "rows"}


class MixtureOfExperts(nn.Module):
    """Logistic router (unnormalised scores of the `top` best) over experts with a clamped gated unit; the score
    multiplies an expert's input.  in_rows = router.  w1 [experts, 2 ff, width] rows [up | gate], w2 [experts, width, ff]."""

    kind = "moe"
    ALPHA, UP_OFFSET = 1.702, 1.0

    def __init__(self, width: int, experts: int, top: int, ff: int, limit: float):
        super().__init__()
        if not 1 <= top <= experts:
            raise ValueError(f"mixture of experts: top={top} of {experts}")
        self.experts, self.top = experts, top
        self.ff = _divide("ff", ff, tp_world_size)
        self.glu = (self.ALPHA, limit, self.UP_OFFSET)
        self.in_rows = experts
        self.w1 = nn.Parameter(torch.empty(experts, 2 * self.ff, width))
        self.w2 = nn.Parameter(torch.empty(experts, width, self.ff))


class GatedResidual(nn.Module):
    """One sublayer with what surrounds it: x <- x + post_norm(sigmoid(gate rows of in_proj(h) + bias) * sublayer(h)),
    h = pre_norm(x)."""

    def __init__(self, width: int, sublayer: nn.Module):
        super().__init__()
        self.width = width
        self.pre_norm = nn.Parameter(torch.ones(width))
        self.post_norm = nn.Parameter(torch.ones(width))
        self.gate_bias = nn.Parameter(torch.zeros(width))
        rows = width + sublayer.in_rows
        self.in_proj = nn.Linear(width, rows + -rows % 8, bias=False)
        self.sublayer = sublayer


MIXERS = {"latent_attention": LatentAttention, "hgrn2": HGRN2}


def make_mixer(kind: str, width: int, m: dict) -> nn.Module:
    """A mixer from its entry in a design's layer list."""
    if kind == "latent_attention":
        rot = m["rot"]
        if rot["dims"] != m["rot_dim"]:
            raise ValueError(f"latent attention: rot.dims={rot['dims']} but rot_dim={m['rot_dim']}")
        return LatentAttention(width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["mask"]["size"],
                               m["scale"], rot["base"])
    if kind == "hgrn2":
        return HGRN2(width, m["heads"], m["dim"], m["vdim"])
    raise ValueError(f"unknown mixer {kind!r}; known: {sorted(MIXERS)}")


def make_mlp(width: int, m: dict) -> nn.Module:
    if m["kind"] != "moe":
        raise ValueError(f"unknown feed-forward {m['kind']!r}; known: ['moe']")
    return MixtureOfExperts(width, m["router"]["experts"], m["router"]["top"], m["expert"]["ff"], m["expert"]["limit"])
