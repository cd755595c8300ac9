"""Sequence mixers of layer-stack models (`models/stack.py`): what a layer does along the sequence axis, each with its
sizes and constants in a spec, its parameters in a module and its per-sequence cache or state in a layout.

  RGLRUMixer              Griffin's recurrent block: short causal convolution, block-diagonal gates, real-gated linear
                          recurrent unit, gelu-gated output
  BiasedWindowAttention   grouped-query attention without rotation: RMS norm over the whole query / key projection,
                          learned bias per (distance bucket, head), sliding window with kept first tokens, sigmoid
                          output gate
  MatrixMemory            mLSTM: matrix memory with exponential input gate, capped gate pre-activations, per-head norm
                          and sigmoid output gate
  ParallelMixer           two mixers on the same input, half the sum of their normed outputs
  TokenShiftMemory        RWKV time mixing: every projection reads its own mix of a token and the one before it, matrix
                          memory with a data-dependent decay per key channel and a bonus for the current token, per-head
                          norm and silu output gate
  ForgetGateMemory        HGRN2: matrix memory whose forget gate (bounded from below) also decides what is written
  RotaryAttention         grouped-query attention with rotary positions (halves of a head or neighbouring dimensions turn
                          together, frequencies may be scaled), RMS-normed query and key heads with or without weights, score
                          cap, sliding window, chunks of positions, a sink in the softmax; may read the keys and values of
                          another layer
  GatedLinearAttention    matrix memory with a decay per key channel, a root of a sigmoid behind a bottleneck; per-head norm
                          and silu output gate
  SumMixer                rotary attention and gated linear attention on the same input, each times a constant, summed
  DistanceAttention       grouped-query attention without rotation: a logarithm of the distance is taken off the scores, value
                          heads are normed, sliding window with kept first tokens, per head a learned sink and an output gate
  LatentAttention         heads of keys and values made from one normed latent per token (which is what is cached), plus one
                          rotated key part that all heads share; sliding window, per head a learned sink

A spec's `kv_rows(dtype)` names the paged cache rows a pass through the layer needs (key columns, value columns), or None
(also for attention that reads another layer's, `kv_from`); `state_shapes()` the fp32 state it keeps per sequence slot. Heads
of attention are stored `stored(dtype)` wide. The kernels are launched by `models/stack_exec.py`.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import ClassVar, NamedTuple, Optional

import torch
import torch.nn as nn

from .transformer import Linear, RMSNorm

MEMORY_SLICE = 32       # value columns a CTA of the matrix-memory kernels owns (csrc/recurrent.cu: MV)
TILE_HEADS = (64, 128, 256)     # head sizes of the tensor-core attention kernels
TILE_PAIRS = ((64, 64), (128, 64), (128, 128), (192, 128), (256, 256))    # (key, value) head sizes of the one for portions
NO_SINK = -math.inf
LATENT_RANK, LATENT_WIDTH = 512, 640    # widest latent, and latent with its rotated part, of the tensor-core decode kernel


def fitted_heads(dim: int, vdim: int, dtype) -> tuple:
    """Widths that heads are stored at: as wide as the tensor-core kernels want them, zeros behind them, where that is bf16 and
    at most twice the size."""
    wide = max(dim, vdim)
    fit = next((w for w in TILE_HEADS if w >= wide), 0)
    return (fit, fit) if dtype == torch.bfloat16 and 0 < fit <= 2 * wide and vdim % 8 == 0 else (dim, vdim)


class YarnScaling(NamedTuple):
    """Rotary frequencies for longer contexts: pairs that turn more than `fast` times over the original context keep theirs,
    those that turn fewer than `slow` times have it divided by the factor, and the pairs between change over linearly; turned
    vectors grow by `size`."""
    factor: float
    original: float
    fast: float
    slow: float

    @property
    def size(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0


# ---------------------------------------------------------------------------------------------------- specs
@dataclass(frozen=True)
class RGLRUSpec:
    width: int
    blocks: int
    conv: int                    # taps of the causal convolution

    def kv_rows(self, dtype):
        return None

    def state_shapes(self) -> dict:
        return {"s": (self.width,), "ring": (self.conv, self.width)}


@dataclass(frozen=True)
class WindowAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: int                # distance from which on every key falls into the last bucket
    window: int                  # 0 = unlimited
    keep_first: int = 0          # leading tokens of the sequence that stay visible
    buckets: int = 32            # rows of the bias table
    chunk: ClassVar[int] = 0
    softcap: ClassVar[float] = 0.0
    sink: ClassVar[float] = NO_SINK

    def stored(self, dtype):
        return self.dim, self.vdim

    def kv_rows(self, dtype):
        return (self.kv_heads * self.dim, self.kv_heads * self.vdim)

    def state_shapes(self) -> dict:
        return {}


@dataclass(frozen=True)
class MatrixMemorySpec:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    def kv_rows(self, dtype):
        return None

    def state_shapes(self) -> dict:
        slices = -(-self.vdim // MEMORY_SLICE)
        return {"S": (self.heads, self.dim, self.vdim), "n": (self.heads, slices, self.dim), "m": (self.heads, slices)}


@dataclass(frozen=True)
class ParallelSpec:
    left: WindowAttentionSpec
    right: MatrixMemorySpec

    def kv_rows(self, dtype):
        return self.left.kv_rows(dtype)

    def state_shapes(self) -> dict:
        return self.right.state_shapes()


@dataclass(frozen=True)
class RotaryAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int                # leading dimensions of a head that turn
    rot_base: float
    softcap: float = 0.0         # scores become softcap * tanh(score / softcap); 0 = as they are
    chunk: int = 0               # a query sees the keys of its own chunk of that many positions; 0 = all before it
    kv_from: Optional[int] = None    # index of the layer whose keys and values this one reads
    window: int = 0              # a query sees itself and the window - 1 keys before it; 0 = all
    interleaved: bool = False    # dimensions 2 i and 2 i + 1 turn together; otherwise i and i + rot_dims / 2
    rot_scaling: Optional[tuple] = None    # (factor, low, high, original context): see stack_exec.rope_frequencies
    head_weights: bool = False   # the norms of query and key heads have weights
    sink: float = NO_SINK        # one more score, without a value, in the sum of the weights
    out_bias: bool = True
    fit_heads: bool = False      # bf16 heads are stored as wide as the tensor-core kernels want them, zeros behind them
    keep_first: ClassVar[int] = 0

    def stored(self, dtype):
        return fitted_heads(self.dim, self.vdim, dtype) if self.fit_heads else (self.dim, self.vdim)

    def kv_rows(self, dtype):
        if self.kv_from is not None:
            return None
        k, v = self.stored(dtype)
        return self.kv_heads * k, self.kv_heads * v

    def state_shapes(self) -> dict:
        return {}


@dataclass(frozen=True)
class TokenShiftMemorySpec:
    heads: int
    dim: int                     # key and value size of a head
    decay_rank: int              # width of the bottleneck that makes the decays
    width: int                   # the mixer's input: the last one of a sequence is part of the state

    def kv_rows(self, dtype):
        return None

    def state_shapes(self) -> dict:
        return {"S": (self.heads, self.dim, self.dim), "last": (self.width,)}


@dataclass(frozen=True)
class ForgetGateMemorySpec:
    heads: int
    dim: int
    vdim: int

    def kv_rows(self, dtype):
        return None

    def state_shapes(self) -> dict:
        return {"S": (self.heads, self.dim, self.vdim)}


@dataclass(frozen=True)
class GatedLinearSpec:
    heads: int
    dim: int
    vdim: int
    tau: float                   # the decay is the tau-th root of a sigmoid
    decay_rank: int              # width of the bottleneck that makes the decays

    def kv_rows(self, dtype):
        return None

    def state_shapes(self) -> dict:
        return {"S": (self.heads, self.dim, self.vdim)}


@dataclass(frozen=True)
class SumSpec:
    left: RotaryAttentionSpec
    right: GatedLinearSpec
    left_scale: float
    right_scale: float

    def kv_rows(self, dtype):
        return self.left.kv_rows(dtype)

    def state_shapes(self) -> dict:
        return self.right.state_shapes()


@dataclass(frozen=True)
class DistanceAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int                  # 0 = unlimited
    keep_first: int = 0          # leading tokens of the sequence that stay visible
    chunk: ClassVar[int] = 0
    softcap: ClassVar[float] = 0.0
    sink: ClassVar[float] = NO_SINK         # the learned ones take its place

    def stored(self, dtype):
        return fitted_heads(self.dim, self.vdim, dtype)

    def kv_rows(self, dtype):
        k, v = self.stored(dtype)
        return self.kv_heads * k, self.kv_heads * v

    def state_shapes(self) -> dict:
        return {}


@dataclass(frozen=True)
class LatentAttentionSpec:
    heads: int
    dim: int                     # unrotated query / key dimensions of a head
    rot_dim: int                 # rotated ones; their key part is shared by all heads
    vdim: int
    kv_rank: int                 # size of the latent
    scale: float
    window: int                  # 0 = unlimited
    rot_dims: int                # leading dimensions of the rotated part that turn
    rot_base: float
    rot_scaling: Optional[tuple] = None     # see stack_exec.rope_frequencies
    kv_heads: ClassVar[int] = 1             # one row of latents serves every head
    chunk: ClassVar[int] = 0
    softcap: ClassVar[float] = 0.0
    sink: ClassVar[float] = NO_SINK
    keep_first: ClassVar[int] = 0

    @property
    def width(self) -> int:
        return self.kv_rank + self.rot_dim

    def tiled(self, dtype) -> bool:
        """Whether the tensor-core kernels take these sizes."""
        return dtype == torch.bfloat16 and not any(n % 8 for n in (self.kv_rank, self.dim, self.rot_dim, self.vdim)) and \
            self.kv_rank <= LATENT_RANK and self.width <= LATENT_WIDTH and self.tile_heads() is not None

    def tile_heads(self) -> Optional[tuple]:
        """Widths of the key and value heads that portions of prompts expand the latents to."""
        return next((p for p in TILE_PAIRS if p[0] >= self.dim + self.rot_dim and p[1] >= self.vdim), None)

    @property
    def split_keys(self) -> bool:
        """Whether the unrotated part of a key fills whole slabs of the tensor-core kernel for portions."""
        return self.dim % 64 == 0

    def stored(self, dtype):
        """Width of a cached row as key and as value: the latent, the rotated part, and zeros up to a multiple of 64."""
        w = -(-self.width // 64) * 64 if self.tiled(dtype) else self.width
        return w, w

    def kv_rows(self, dtype):
        return self.stored(dtype)[0], 0

    def state_shapes(self) -> dict:
        return {}


# ------------------------------------------------------------------------------------------------- bias table
def distance_buckets(rows: int, bias_max: int, device=None) -> torch.Tensor:
    """Bucket of every distance 0 .. bias_max: the lower half of the rows holds one distance each, the upper half
    grows logarithmically and ends at `bias_max`; larger distances share the last row with it."""
    half = rows // 2
    n = torch.arange(bias_max + 1, dtype=torch.float64, device=device)
    if half < 1 or bias_max <= half:
        return torch.clamp(n, max=rows - 1).long()
    log_pos = torch.log(torch.clamp(n, min=1) / half) / math.log(bias_max / half) * (rows - half)
    # a ratio that is an integer in exact arithmetic must not fall below it by rounding
    upper = torch.clamp(half + torch.floor(log_pos + 1e-12), max=rows - 1)
    return torch.where(n < half, n, upper).long()


# --------------------------------------------------------------------------------------------------- modules
def _param(*shape, dtype, device, fill: float = 0.0):
    return nn.Parameter(torch.full(shape, fill, dtype=dtype, device=device))


class RGLRUMixer(nn.Module):
    def __init__(self, spec: RGLRUSpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        if spec.width % spec.blocks:
            raise ValueError(f"{spec.width} channels do not split into {spec.blocks} blocks")
        self.spec = spec
        W, bs = spec.width, spec.width // spec.blocks
        self.y_proj = Linear(width, W, True, dtype, device)
        self.x_proj = Linear(width, W, True, dtype, device)
        self.conv_weight = _param(W, spec.conv, dtype=dtype, device=device)
        self.conv_bias = _param(W, dtype=dtype, device=device)
        self.ra_weight = _param(spec.blocks, bs, bs, dtype=dtype, device=device)
        self.ra_bias = _param(spec.blocks, bs, dtype=dtype, device=device)
        self.ri_weight = _param(spec.blocks, bs, bs, dtype=dtype, device=device)
        self.ri_bias = _param(spec.blocks, bs, dtype=dtype, device=device)
        self.lam = _param(W, dtype=dtype, device=device, fill=-4.0)
        self.o_proj = Linear(W, width, False, dtype, device)

    def init_special(self) -> None:
        self.conv_weight.zero_()
        self.conv_weight[:, -1] = 1.0
        self.ra_bias.zero_()
        self.ri_bias.zero_()

    def fused_groups(self) -> list:
        return [[self.y_proj, self.x_proj]]


class BiasedWindowAttention(nn.Module):
    def __init__(self, spec: WindowAttentionSpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        if spec.heads % spec.kv_heads:
            raise ValueError(f"{spec.heads} query heads over {spec.kv_heads} key / value heads")
        self.spec, self.eps = spec, eps
        H, G = spec.heads, spec.kv_heads
        self.q_proj = Linear(width, H * spec.dim, False, dtype, device)
        self.k_proj = Linear(width, G * spec.dim, False, dtype, device)
        self.v_proj = Linear(width, G * spec.vdim, False, dtype, device)
        self.g_proj = Linear(width, H * spec.vdim, False, dtype, device)
        self.o_proj = Linear(H * spec.vdim, width, False, dtype, device)
        self.q_norm = RMSNorm(H * spec.dim, eps, False, dtype, device)
        self.k_norm = RMSNorm(G * spec.dim, eps, False, dtype, device)
        self.rel = _param(spec.buckets, H, dtype=dtype, device=device)

    def bias_table(self) -> torch.Tensor:
        """fp32 [heads, far + 1]: what is added to the score of a key at distance min(i - j, far)."""
        idx = distance_buckets(self.rel.shape[0], self.spec.bias_max, self.rel.device)
        return self.rel.detach().float()[idx].t().contiguous()

    def init_special(self) -> None:
        pass


class MatrixMemory(nn.Module):
    def __init__(self, spec: MatrixMemorySpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        self.spec, self.eps = spec, eps
        H = spec.heads
        self.q_proj = Linear(width, H * spec.dim, False, dtype, device)
        self.k_proj = Linear(width, H * spec.dim, False, dtype, device)
        self.v_proj = Linear(width, H * spec.vdim, False, dtype, device)
        self.g_proj = Linear(width, H * spec.vdim, False, dtype, device)
        self.i_proj = Linear(width, H, True, dtype, device)
        self.f_proj = Linear(width, H, True, dtype, device)
        self.o_proj = Linear(H * spec.vdim, width, False, dtype, device)
        self.norm = RMSNorm(H * spec.vdim, eps, False, dtype, device)

    def init_special(self) -> None:
        self.f_proj.bias.fill_(3.0)


class ParallelMixer(nn.Module):
    def __init__(self, spec: ParallelSpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        self.spec = spec
        self.left = BiasedWindowAttention(spec.left, width, eps, dtype, device)
        self.right = MatrixMemory(spec.right, width, eps, dtype, device)
        self.left_norm = RMSNorm(width, eps, False, dtype, device)
        self.right_norm = RMSNorm(width, eps, False, dtype, device)

    def init_special(self) -> None:
        self.left.init_special()
        self.right.init_special()

    def fused_groups(self) -> list:
        lf, rt = self.left, self.right
        return [[lf.q_proj, lf.k_proj, lf.v_proj, lf.g_proj, rt.q_proj, rt.k_proj, rt.v_proj, rt.g_proj],
                [rt.i_proj, rt.f_proj]]


class RotaryAttention(nn.Module):
    def __init__(self, spec: RotaryAttentionSpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        if spec.heads % spec.kv_heads:
            raise ValueError(f"{spec.heads} query heads over {spec.kv_heads} key / value heads")
        if spec.rot_dims % 2 or spec.rot_dims > spec.dim:
            raise ValueError(f"{spec.rot_dims} rotated dimensions of {spec.dim}")
        self.spec, self.eps = spec, eps
        self.q_proj = Linear(width, spec.heads * spec.dim, True, dtype, device)
        own = spec.kv_from is None
        self.k_proj = Linear(width, spec.kv_heads * spec.dim, True, dtype, device) if own else None
        self.v_proj = Linear(width, spec.kv_heads * spec.vdim, True, dtype, device) if own else None
        self.o_proj = Linear(spec.heads * spec.vdim, width, spec.out_bias, dtype, device)
        self.q_norm = RMSNorm(spec.dim, eps, False, dtype, device) if spec.head_weights else None
        self.k_norm = RMSNorm(spec.dim, eps, False, dtype, device) if spec.head_weights and own else None

    def init_special(self) -> None:
        pass

    def fused_groups(self) -> list:
        return [[self.q_proj] + ([self.k_proj, self.v_proj] if self.k_proj is not None else [])]


class TokenShiftMemory(nn.Module):
    MIXES = ("r", "k", "v", "g", "w")

    def __init__(self, spec: TokenShiftMemorySpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        self.spec, self.eps = spec, eps
        C = spec.heads * spec.dim
        for n in self.MIXES:
            setattr(self, "mu_" + n, _param(width, dtype=dtype, device=device, fill=0.5))
        for n in ("r", "k", "v", "g"):
            setattr(self, n + "_proj", Linear(width, C, False, dtype, device))
        self.w1_proj = Linear(width, spec.decay_rank, False, dtype, device)
        self.w2_proj = Linear(spec.decay_rank, C, False, dtype, device)
        self.w0 = _param(C, dtype=dtype, device=device)
        self.u = _param(spec.heads, spec.dim, dtype=dtype, device=device)
        self.norm = RMSNorm(C, eps, False, dtype, device)
        self.o_proj = Linear(C, width, False, dtype, device)

    def mu(self) -> torch.Tensor:
        return torch.stack([getattr(self, "mu_" + n).data for n in self.MIXES])

    def init_special(self) -> None:
        n = self.w0.numel()
        self.w0.copy_(torch.linspace(-6.0, 0.0, n, device=self.w0.device))      # slow to fast decays over the channels

    def fused_groups(self) -> list:
        return []


class ForgetGateMemory(nn.Module):
    def __init__(self, spec: ForgetGateMemorySpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        self.spec, self.eps = spec, eps
        self.q_proj = Linear(width, spec.heads * spec.dim, False, dtype, device)
        self.v_proj = Linear(width, spec.heads * spec.vdim, False, dtype, device)
        self.f_proj = Linear(width, spec.heads * spec.dim, True, dtype, device)
        self.lower = _param(spec.heads * spec.dim, dtype=dtype, device=device, fill=0.5)
        self.norm = RMSNorm(spec.vdim, eps, False, dtype, device)
        self.o_proj = Linear(spec.heads * spec.vdim, width, False, dtype, device)

    def init_special(self) -> None:
        self.f_proj.bias.fill_(2.0)

    def fused_groups(self) -> list:
        return [[self.q_proj, self.v_proj], [self.f_proj]]


class GatedLinearAttention(nn.Module):
    def __init__(self, spec: GatedLinearSpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        self.spec, self.eps = spec, eps
        K, C = spec.heads * spec.dim, spec.heads * spec.vdim
        self.q_proj = Linear(width, K, False, dtype, device)
        self.k_proj = Linear(width, K, False, dtype, device)
        self.v_proj = Linear(width, C, False, dtype, device)
        self.g_proj = Linear(width, C, False, dtype, device)
        self.a1_proj = Linear(width, spec.decay_rank, False, dtype, device)
        self.a2_proj = Linear(spec.decay_rank, K, True, dtype, device)
        self.norm = RMSNorm(spec.vdim, eps, False, dtype, device)
        self.o_proj = Linear(C, width, False, dtype, device)

    def init_special(self) -> None:
        self.a2_proj.bias.fill_(2.0)

    def fused_groups(self) -> list:
        return [[self.q_proj, self.k_proj, self.v_proj, self.g_proj, self.a1_proj]]


class SumMixer(nn.Module):
    def __init__(self, spec: SumSpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        if spec.left.out_bias or spec.left.kv_from is not None:
            raise ValueError("attention beside another mixer has keys of its own and no output bias")
        self.spec = spec
        self.left = RotaryAttention(spec.left, width, eps, dtype, device)
        self.right = GatedLinearAttention(spec.right, width, eps, dtype, device)

    def init_special(self) -> None:
        self.left.init_special()
        self.right.init_special()

    def fused_groups(self) -> list:
        return [self.left.fused_groups()[0] + self.right.fused_groups()[0]]


class DistanceAttention(nn.Module):
    def __init__(self, spec: DistanceAttentionSpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        if spec.heads % spec.kv_heads:
            raise ValueError(f"{spec.heads} query heads over {spec.kv_heads} key / value heads")
        self.spec, self.eps = spec, eps
        H, G = spec.heads, spec.kv_heads
        self.q_proj = Linear(width, H * spec.dim, False, dtype, device)
        self.k_proj = Linear(width, G * spec.dim, False, dtype, device)
        self.v_proj = Linear(width, G * spec.vdim, False, dtype, device)
        self.g_proj = Linear(width, H, False, dtype, device)
        self.o_proj = Linear(H * spec.vdim, width, False, dtype, device)
        self.r1 = _param(H, dtype=dtype, device=device, fill=1.0)
        self.r2 = _param(H, dtype=dtype, device=device, fill=1.0)
        self.sink = _param(H, dtype=dtype, device=device)

    def bias_table(self, positions: int) -> torch.Tensor:
        """fp32 [heads, positions]: what is added to the score of a key at every distance, -r1 ln(1 + r2 distance)."""
        r1, r2 = (r.detach().double()[:, None] for r in (self.r1, self.r2))
        gap = torch.arange(positions, dtype=torch.float64, device=r1.device)
        return (-r1 * torch.log1p(r2 * gap)).float()

    def init_special(self) -> None:
        self.r1.fill_(1.0)
        self.r2.fill_(1.0)

    def fused_groups(self) -> list:
        return [[self.q_proj, self.k_proj, self.v_proj, self.g_proj]]


class LatentAttention(nn.Module):
    def __init__(self, spec: LatentAttentionSpec, width: int, eps: float, dtype, device=None):
        super().__init__()
        if spec.rot_dims % 2 or spec.rot_dims > spec.rot_dim:
            raise ValueError(f"{spec.rot_dims} rotated dimensions of {spec.rot_dim}")
        self.spec, self.eps = spec, eps
        H = spec.heads
        self.q_proj = Linear(width, H * (spec.dim + spec.rot_dim), False, dtype, device)
        self.dkv_proj = Linear(width, spec.width, False, dtype, device)
        self.kv_norm = RMSNorm(spec.kv_rank, eps, False, dtype, device)
        self.uk_proj = Linear(spec.kv_rank, H * spec.dim, False, dtype, device)
        self.uv_proj = Linear(spec.kv_rank, H * spec.vdim, False, dtype, device)
        self.o_proj = Linear(H * spec.vdim, width, False, dtype, device)
        self.sink = _param(H, dtype=dtype, device=device)

    @torch.no_grad()
    def expansion(self, stored: int) -> torch.Tensor:
        """What takes a cached row to the heads' keys and behind all of them to their values, as the attention kernel of portions
        reads them. Keys of whole slabs of 64 are made from the latent alone, [heads * (dim + value width), rank]: the kernel reads the
        shared rotated part from the cached rows themselves. Otherwise [heads * (key width + value width), stored]: a key is made
        from the latent, then the rotated part, then zeros."""
        sp, H = self.spec, self.spec.heads
        wide, wide_v = sp.tile_heads()
        if sp.split_keys:
            w = self.uk_proj.weight.new_zeros(H * (sp.dim + wide_v), sp.kv_rank)
            w[:H * sp.dim] = self.uk_proj.weight
            w[H * sp.dim:].view(H, wide_v, sp.kv_rank)[:, :sp.vdim] = self.uv_proj.weight.view(H, sp.vdim, sp.kv_rank)
            return w
        w = self.uk_proj.weight.new_zeros(H * (wide + wide_v), stored)
        k, v = w[:H * wide].view(H, wide, stored), w[H * wide:].view(H, wide_v, stored)
        k[:, :sp.dim, :sp.kv_rank] = self.uk_proj.weight.view(H, sp.dim, sp.kv_rank)
        k[:, sp.dim:sp.dim + sp.rot_dim, sp.kv_rank:sp.width] = torch.eye(sp.rot_dim, dtype=w.dtype, device=w.device)
        v[:, :sp.vdim, :sp.kv_rank] = self.uv_proj.weight.view(H, sp.vdim, sp.kv_rank)
        return w

    def init_special(self) -> None:
        pass

    def fused_groups(self) -> list:
        return [[self.q_proj, self.dkv_proj]]


MIXERS = {DistanceAttentionSpec: DistanceAttention, LatentAttentionSpec: LatentAttention, RGLRUSpec: RGLRUMixer, ParallelSpec: ParallelMixer, RotaryAttentionSpec: RotaryAttention,
          TokenShiftMemorySpec: TokenShiftMemory, ForgetGateMemorySpec: ForgetGateMemory, GatedLinearSpec: GatedLinearAttention,
          SumSpec: SumMixer}


def create_mixer(spec, width: int, eps: float, dtype, device: Optional[torch.device] = None) -> nn.Module:
    return MIXERS[type(spec)](spec, width, eps, dtype, device)
