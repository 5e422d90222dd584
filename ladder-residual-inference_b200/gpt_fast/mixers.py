"""Sublayers of layer-list designs: latent attention, chunked grouped-query attention, the HGRN2 recurrence, gated linear
attention, the gated delta rule, two mixers side by side, a mixture of experts and a dense gated unit, with the caches they
keep; and the two ways a sublayer sits in the residual (`GatedResidual`, `StreamBranch`).  Beside the Llama sublayers of `utils`, with every size and constant a constructor argument.

Modules own parameters and cache buffers in the layout the kernels read; `engine_layers.LayerEngine` runs them.
Tensor parallelism is fixed at construction as everywhere in the package: heads and expert widths are divided by the
world size, projections from the model width are split by rows, projections back to it by columns.

A sublayer's input projections are fused into one, with the projection of the gate that scales its result where there is
one (see `GatedResidual`): `in_proj` rows = [gate (width) | sublayer rows | zero rows up to a multiple of 8].
"""
import math
from typing import Dict, List, NamedTuple

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


class GroupedKVCache(nn.Module):
    """Keys [max_batch, kv_heads, max_seq, dim] and values [max_batch, kv_heads, max_seq, vdim]."""

    def __init__(self, max_batch_size, max_seq_length, kv_heads, dim, vdim, dtype):
        super().__init__()
        self.register_buffer("k_cache", torch.zeros(max_batch_size, kv_heads, max_seq_length, dim, dtype=dtype))
        self.register_buffer("v_cache", torch.zeros(max_batch_size, kv_heads, max_seq_length, vdim, dtype=dtype))


class ConvState(nn.Module):
    """fp32 ring [max_batch, taps, channels] of convolution inputs: position p in slot p % taps.  Positions before the
    sequence's start are never read, so a call at position 0 needs no reset."""

    def __init__(self, max_batch_size, taps, channels):
        super().__init__()
        self.register_buffer("ring", torch.zeros(max_batch_size, taps, channels, dtype=torch.float32))


class Rows(NamedTuple):
    """Rows of an input projection: checkpoint tensor, how it is split over ranks ("rows" or "all"), rows on a rank, and the
    rows they take with zero rows behind them."""
    name: str
    split: str
    rows: int
    padded: int


def _padded(n: int) -> int:
    return n + -n % 8


def _offsets(parts: List[Rows], start: int = 0) -> Dict[str, int]:
    """First row of every part."""
    out = {}
    for p in parts:
        out[p.name] = start
        start += p.padded
    return out


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


class ChunkedAttention(nn.Module):
    """Grouped-query attention inside chunks of positions (and / or a sliding window), with RMSNorm over the whole query and
    key projections, rotation of the first rot_dims dimensions of a head, and a learned logit per head (`sink`) that joins
    the softmax denominator."""

    kind = "chunked_attention"

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, rot_dims: int, rot_base: float, chunk: int = 0,
                 window: int = 0):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"chunked attention: {heads} heads do not share {kv_heads} key heads evenly")
        if rot_dims % 2 or not 0 <= rot_dims <= dim:
            raise ValueError(f"chunked attention: {rot_dims} rotated dimensions of {dim}")
        if chunk < 0 or window < 0:
            raise ValueError(f"chunked attention: chunk={chunk} window={window}")
        self.heads, self.kv_heads = _divide("heads", heads, tp_world_size), _divide("kv_heads", kv_heads, tp_world_size)
        self.dim, self.vdim, self.scale = dim, vdim, scale
        self.rot_dims, self.rot_base, self.chunk, self.window = rot_dims, rot_base, chunk, window
        self.norm_widths = (heads * dim, kv_heads * dim)  # over all ranks
        self.q_norm = nn.Parameter(torch.ones(self.heads * dim))
        self.k_norm = nn.Parameter(torch.ones(self.kv_heads * dim))
        self.sink = nn.Parameter(torch.zeros(self.heads))
        self.kv_cache = None

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def parts(self) -> List[Rows]:
        q, k, v = self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim
        return [Rows("q", "rows", q, q), Rows("k", "rows", k, k), Rows("v", "rows", v, v)]

    def setup_cache(self, max_batch, max_seq, dtype, device):
        self.kv_cache = GroupedKVCache(max_batch, max_seq, self.kv_heads, self.dim, self.vdim, dtype).to(device)
        self.rope_table = rotate_half_table(max_seq, max(self.rot_dims, 2), self.rot_base, device)

    def recurrent_state(self) -> List[Tensor]:
        return []


class GatedDelta(nn.Module):
    """Gated delta rule: short convolutions on q, k, v, unit queries and keys, a decay per key channel and a gate on the
    normed result, both from low-rank projections.  Ranks are padded to multiples of 8 with zeros."""

    kind = "gated_delta"

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, decay_rank: int, gate_rank: int):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"gated delta rule: {heads} heads do not share {kv_heads} key heads evenly")
        if taps < 1:
            raise ValueError(f"gated delta rule: {taps} convolution taps")
        self.heads, self.kv_heads = _divide("heads", heads, tp_world_size), _divide("kv_heads", kv_heads, tp_world_size)
        self.dim, self.vdim, self.taps = dim, vdim, taps
        self.decay_rank, self.gate_rank = decay_rank, gate_rank
        qk, hc, he = self.kv_heads * dim, self.heads * dim, self.heads * vdim
        self.conv_q = nn.Parameter(torch.empty(qk, taps))
        self.conv_k = nn.Parameter(torch.empty(qk, taps))
        self.conv_v = nn.Parameter(torch.empty(he, taps))
        self.a2 = nn.Parameter(torch.empty(hc, _padded(decay_rank)))
        self.g2 = nn.Parameter(torch.empty(he, _padded(gate_rank)))
        self.a_log = nn.Parameter(torch.zeros(self.heads))
        self.dt_bias = nn.Parameter(torch.zeros(hc))
        self.norm = nn.Parameter(torch.ones(vdim))
        self.kv_cache = None

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def parts(self) -> List[Rows]:
        qk, v = self.kv_heads * self.dim, self.heads * self.vdim
        return [Rows("q", "rows", qk, qk), Rows("k", "rows", qk, qk), Rows("v", "rows", v, v),
                Rows("a1", "all", self.decay_rank, _padded(self.decay_rank)),
                Rows("g1", "all", self.gate_rank, _padded(self.gate_rank)), Rows("b", "rows", self.heads, self.heads)]

    def setup_cache(self, max_batch, max_seq, dtype, device):
        self.kv_cache = RecurrentState(max_batch, self.heads, self.dim, self.vdim).to(device)
        self.conv_state = ConvState(max_batch, self.taps, 2 * self.kv_heads * self.dim + self.heads * self.vdim).to(device)

    def recurrent_state(self) -> List[Tensor]:
        return [self.kv_cache.state, self.conv_state.ring]


class ParallelMixers(nn.Module):
    """Two mixers that read the same input; their results are weighted, and projected by one matrix [left o | right o]."""

    kind = "parallel"

    def __init__(self, width: int, left: nn.Module, right: nn.Module, left_scale: float, right_scale: float):
        super().__init__()
        self.left, self.right, self.scales = left, right, (left_scale, right_scale)
        self.wo = nn.Linear(self.out_width, width, bias=False)

    @property
    def out_width(self) -> int:
        return self.left.out_width + self.right.out_width

    @property
    def in_rows(self) -> int:
        return sum(p.padded for p in self.parts())

    def parts(self) -> List[Rows]:
        return [p._replace(name=f"{side}.{p.name}") for side, m in (("left", self.left), ("right", self.right)) for p in m.parts()]

    def setup_cache(self, max_batch, max_seq, dtype, device):
        self.left.setup_cache(max_batch, max_seq, dtype, device)
        self.right.setup_cache(max_batch, max_seq, dtype, device)

    def recurrent_state(self) -> List[Tensor]:
        return self.left.recurrent_state() + self.right.recurrent_state()


class GatedLinearAttention(nn.Module):
    """Linear attention with a decay sigmoid(z)^(1 / tau) per key channel, z from a low-rank projection (rank padded to a
    multiple of 8 with zeros), and a silu gate on the normed result."""

    kind = "gla"

    def __init__(self, width: int, heads: int, dim: int, vdim: int, tau: float, decay_rank: int):
        super().__init__()
        self.heads = _divide("heads", heads, tp_world_size)
        self.dim, self.vdim, self.tau, self.decay_rank = dim, vdim, tau, decay_rank
        self.a2 = nn.Parameter(torch.empty(self.heads * dim, _padded(decay_rank)))
        self.a2_bias = nn.Parameter(torch.zeros(self.heads * dim))
        self.norm = nn.Parameter(torch.ones(vdim))
        self.wo = nn.Linear(self.heads * vdim, width, bias=False)
        self.kv_cache = None

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def in_rows(self) -> int:
        return sum(p.padded for p in self.parts())

    def parts(self) -> List[Rows]:
        qk, v = self.heads * self.dim, self.heads * self.vdim
        return [Rows("q", "rows", qk, qk), Rows("k", "rows", qk, qk), Rows("v", "rows", v, v), Rows("g", "rows", v, v),
                Rows("a1", "all", self.decay_rank, _padded(self.decay_rank))]

    def setup_cache(self, max_batch, max_seq, dtype, device):
        self.kv_cache = RecurrentState(max_batch, self.heads, self.dim, self.vdim).to(device)

    def recurrent_state(self) -> List[Tensor]:
        return [self.kv_cache.state]


class DenseGLU(nn.Module):
    """Clamped gated unit, g sigmoid(alpha g) (u + offset) with g = min(gate, limit), u = clamp(up, -limit, limit).
    w1 [2 ff, width] rows [up | gate], w2 [width, ff]."""

    kind = "glu"
    ALPHA, UP_OFFSET = 1.702, 1.0
    in_rows = 0

    def __init__(self, width: int, ff: int, limit: float):
        super().__init__()
        self.ff = _divide("ff", ff, tp_world_size)
        self.glu = (self.ALPHA, limit, self.UP_OFFSET)
        self.w1 = nn.Parameter(torch.empty(2 * self.ff, width))
        self.w2 = nn.Parameter(torch.empty(width, self.ff))


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
        self.width = self.gate_rows = width
        self.pre_norm = nn.Parameter(torch.ones(width))
        self.post_norm = nn.Parameter(torch.ones(width))
        self.gate_bias = nn.Parameter(torch.zeros(width))
        rows = width + sublayer.in_rows
        self.in_proj = nn.Linear(width, rows + -rows % 8, bias=False)
        self.sublayer = sublayer


class StreamBranch(nn.Module):
    """One sublayer over a residual of several streams x_1 .. x_n: y = sublayer(norm(sum_s in[s] x_s)), then
    x_t <- sum_s mix[s, t] x_s + out[t] y."""

    def __init__(self, width: int, streams: int, sublayer: nn.Module):
        super().__init__()
        self.width, self.gate_rows = width, 0
        self.pre_norm = nn.Parameter(torch.ones(width))
        self.w_in = nn.Parameter(torch.ones(streams))
        self.w_mix = nn.Parameter(torch.eye(streams))
        self.w_out = nn.Parameter(torch.ones(streams))
        self.in_proj = nn.Linear(width, _padded(sublayer.in_rows), bias=False) if sublayer.in_rows else None
        self.sublayer = sublayer


MIXERS = {"latent_attention": LatentAttention, "hgrn2": HGRN2, "parallel": ParallelMixers, "gla": GatedLinearAttention}


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
    if kind == "gla":
        return GatedLinearAttention(width, m["heads"], m["dim"], m["vdim"], m["tau"], m["decay_rank"])
    if kind == "parallel":
        a, b = m["left"], m["right"]
        left = ChunkedAttention(a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], a["rot"]["dims"], a["rot"]["base"],
                                chunk=a["mask"]["size"])
        right = GatedDelta(b["heads"], b["kv_heads"], b["dim"], b["vdim"], b["conv"], b["decay_rank"], b["gate_rank"])
        return ParallelMixers(width, left, right, m["left_scale"], m["right_scale"])
    raise ValueError(f"unknown mixer {kind!r}; known: {sorted(MIXERS)}")


def make_mlp(width: int, m: dict) -> nn.Module:
    if m["kind"] == "dense":
        return DenseGLU(width, m["ff"], m["limit"])
    if m["kind"] != "moe":
        raise ValueError(f"unknown feed-forward {m['kind']!r}; known: ['dense', 'moe']")
    return MixtureOfExperts(width, m["router"]["experts"], m["router"]["top"], m["expert"]["ff"], m["expert"]["limit"])
