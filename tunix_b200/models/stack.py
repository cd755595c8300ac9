"""Layer-stack models: decoders whose layers are listed one by one, each with its own mixer (`models/mixers.py`) and
feed-forward, a range of layers that may run several times with the same weights, parallel residual streams joined by
hyper-connections, norms over groups of a row and behind sublayers, learned position rows, mixtures of experts, and inputs per
token and layer. Designs of this kind: Roluzen, Tovalix, Zikezen, Zigipel.

The residual streams are fp32. A sublayer q of a layer reads u = sum_s in[s] x_s, computes y = f(norm(u)) and leaves
x_t = sum_s mix[s, t] x_s + out[t] y on every stream (`post_norms`: y is normed once more); the model's output is the norm of
the streams' sum. With `loop_embed` the embedding output is added again before every pass of the loop but the first; with
`loop_input` every pass t begins with x = W [x; embedding output] + step_t. A layer's token input adds
norm(proj(gelu(gate(x)) * e)) after the feed-forward, e being the layer's part of the token's row in a second embedding table.
With `parallel_ff` mixer and feed-forward of a layer read the same norm and are added together; with `token_shift` a mixer reads
h + (row before - h) * mu instead of h. The embedding may add a row per pair of neighbouring tokens (`bigram`).

The model holds parameters; `models/stack_exec.py` runs it on ragged batches over the paged cache and the slot states of
`generate/engine.py`. `forward` scores whole sequences through that same path on a temporary cache (no gradients).
"""
from __future__ import annotations

import dataclasses
import json
import os
from dataclasses import dataclass, field
from typing import Optional, Union

import torch
import torch.nn as nn

from ..ops import functional as F
from .config import ModelConfig
from .mixers import (DistanceAttentionSpec, ForgetGateMemorySpec, GatedLinearSpec, LatentAttentionSpec, MatrixMemorySpec, ParallelSpec,
                     RGLRUSpec, RotaryAttentionSpec, SumSpec, TokenShiftMemorySpec, WindowAttentionSpec, YarnScaling, create_mixer)
from .transformer import MLP, Linear, RMSNorm


@dataclass(frozen=True)
class LayerSpec:
    mixer: object                       # one of the specs of models/mixers.py
    ff: Optional[int]                   # width of the feed-forward (of an expert); None = the layer has none
    ff_kind: str = "glu"                # "glu": gated by the model's activation; "xielu": up, xIELU with two learned numbers, down; "experts"
    experts: int = 0                    # silu-gated experts, of which a token uses `top`
    top: int = 0


@dataclass
class StackConfig(ModelConfig):
    layer_specs: tuple = field(default_factory=tuple)
    loop: Optional[tuple] = None        # (start, stop, times): these layers run `times` times in a row
    streams: int = 0                    # residual streams with hyper-connections; 0 = one plain residual
    norm_groups: int = 1                # equal parts of a row that the norms before sublayers and at the ends are taken over
    embed_norm: bool = False            # the embedding rows are normed
    token_side: int = 0                 # width of the per-layer token inputs; 0 = none
    embed_factor: float = 1.0           # of the embedding rows
    positions: int = 0                  # rows of the learned position table, the longest sequence; 0 = no table
    loop_embed: bool = False            # the embedding output is added again before each pass of the loop but the first
    loop_input: bool = False            # each pass of the loop begins with a product of [x; embedding output] and a vector of its own
    bigram: Optional[tuple] = None      # (buckets, factor of the token before, factor of the token): hashed rows of token pairs
    parallel_ff: bool = False           # mixer and feed-forward of a layer read the same norm
    token_shift: bool = False           # mixers read a mix of a token's normed row and the one before it
    ff_bias: bool = False               # biases of the feed-forward's projections
    logit_scale: float = 1.0

    def __post_init__(self):
        if not self.layer_specs:
            raise ValueError("a layer-stack model needs its layers")
        self.num_layers = len(self.layer_specs)
        ffs = [s.ff for s in self.layer_specs if s.ff is not None]
        self.hidden_dim = max(ffs) if ffs else 0
        att = [getattr(s.mixer, "left", s.mixer) for s in self.layer_specs]
        att = [a for a in att if isinstance(a, (WindowAttentionSpec, RotaryAttentionSpec, DistanceAttentionSpec, LatentAttentionSpec))]
        if att:                         # what generic callers size caches and reports by: the first attention layer
            self.num_heads, self.num_kv_heads, self.head_dim = att[0].heads, att[0].kv_heads, att[0].dim
        if self.loop is not None:
            a, b, times = self.loop
            if not (0 <= a <= b <= self.num_layers and times >= 0):
                raise ValueError(f"loop {self.loop} does not fit {self.num_layers} layers")
        if self.parallel_ff and (self.post_norms or self.streams or self.token_side):
            raise ValueError("layers whose sublayers run side by side have one plain residual and no norms behind sublayers")
        if (self.parallel_ff or self.token_shift) and not all(
                isinstance(s.mixer, (DistanceAttentionSpec, LatentAttentionSpec)) and s.ff_kind == "glu" for s in self.layer_specs):
            raise ValueError("this layer form takes distance or latent attention and gated feed-forwards")
        if self.parallel_ff != self.token_shift:
            raise ValueError("shifted mixers and side by side sublayers come together")
        if self.logit_scale == 0.0 or (self.logit_scale != 1.0 and self.final_logit_softcap):
            raise ValueError(f"a logit scale of {self.logit_scale}" + (" beside a score cap" if self.final_logit_softcap else ""))
        if self.embed_dim % self.norm_groups:
            raise ValueError(f"a width of {self.embed_dim} does not split into {self.norm_groups} norm groups")
        for i, s in enumerate(self.layer_specs):
            if s.ff_kind == "experts" and s.ff is not None and not 1 <= s.top <= s.experts:
                raise ValueError(f"layer {i}: {s.top} of {s.experts} experts")
            if self.post_norms and isinstance(s.mixer, ParallelSpec):
                raise ValueError(f"layer {i}: the halves of this mixer are normed already")
            j = getattr(s.mixer, "kv_from", None)
            if j is None:
                continue
            src = self.layer_specs[j].mixer if 0 <= j < i else None
            if not isinstance(src, RotaryAttentionSpec) or src.kv_from is not None:
                raise ValueError(f"layer {i} reads keys and values of layer {j}, which keeps none before it")
            if (src.kv_heads, src.dim, src.vdim) != (s.mixer.kv_heads, s.mixer.dim, s.mixer.vdim):
                raise ValueError(f"layers {i} and {j} share keys and values of unequal sizes")
        self.kv_sources()

    def runs(self) -> list:
        """Layer index of every pass, in order. Each pass has its own cache and state."""
        n = self.num_layers
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    def restarts(self) -> set:
        """The passes (indices into `runs`) that begin a repetition of the loop."""
        if self.loop is None:
            return set()
        a, b, times = self.loop
        return {a + t * (b - a) for t in range(1, times)} if b > a else set()

    def loop_starts(self) -> dict:
        """Pass (index into `runs`) -> number of the loop's repetition that it begins."""
        if self.loop is None:
            return {}
        a, b, times = self.loop
        return {a + t * (b - a): t for t in range(times)} if b > a else {}

    # ---- what the engine's cache manager allocates, per pass
    def kv_rows(self, dtype: Optional[torch.dtype] = None) -> list:
        return [self.layer_specs[i].mixer.kv_rows(dtype or self.dtype) for i in self.runs()]

    def kv_sources(self) -> list:
        """Per pass, the pass whose cache its attention reads: its own, or the last pass of the layer it shares with."""
        last, out = {}, []
        for r, i in enumerate(self.runs()):
            j = getattr(self.layer_specs[i].mixer, "kv_from", None)
            if j is not None and j not in last:
                raise ValueError(f"layer {i} reads keys and values of layer {j}, which has not run before it")
            out.append(r if j is None else last[j])
            last[i] = r
        return out

    def state_shapes(self) -> list:
        before = {"before": (self.embed_dim,)} if self.token_shift else {}     # the normed row of the sequence's last token
        return [{**self.layer_specs[i].mixer.state_shapes(), **before} for i in self.runs()]

    def token_states(self) -> tuple:
        """Token ids that a sequence keeps besides the states of its layer passes."""
        return ("last",) if self.bigram else ()

    def num_params(self) -> int:
        return sum(p.numel() for p in StackModel(self, device=torch.device("meta")).parameters())

    # ---- presets (random weights: no checkpoint of this design is published)
    @classmethod
    def roluzen_tiny(cls) -> "StackConfig":
        att = WindowAttentionSpec(heads=4, kv_heads=2, dim=32, vdim=32, scale=32 ** -0.5, bias_max=64, window=24, keep_first=2,
                                  buckets=12)
        par = LayerSpec(ParallelSpec(att, MatrixMemorySpec(heads=2, dim=24, vdim=40, gate_cap=12.0)), 192)
        rec = LayerSpec(RGLRUSpec(width=160, blocks=5, conv=4), 192)
        return cls(family="roluzen", vocab_size=384, embed_dim=128, layer_specs=(rec, par, rec), loop=(1, 3, 2), streams=3)

    @classmethod
    def _roluzen(cls, D, ff, heads, kv, dim, mh, mdk, mdv, W, blocks, n, loop, window=1024, vocab=151936):
        att = WindowAttentionSpec(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, bias_max=4 * window,
                                  window=window, keep_first=4, buckets=32)
        par = LayerSpec(ParallelSpec(att, MatrixMemorySpec(heads=mh, dim=mdk, vdim=mdv, gate_cap=15.0)), ff)
        rec = LayerSpec(RGLRUSpec(width=W, blocks=blocks, conv=4), ff)
        specs = tuple(par if i % 3 == 0 else rec for i in range(n))
        return cls(family="roluzen", vocab_size=vocab, embed_dim=D, layer_specs=specs, loop=loop, streams=2)

    @classmethod
    def roluzen_2b(cls) -> "StackConfig":
        return cls._roluzen(2048, 6144, 16, 8, 128, 8, 128, 256, 2048, 16, 18, (0, 3, 2))

    @classmethod
    def roluzen_8b(cls) -> "StackConfig":
        return cls._roluzen(4096, 12288, 32, 8, 128, 8, 256, 512, 4096, 16, 24, (0, 3, 2))

    @classmethod
    def _tovalix(cls, D, ff, heads, kv, dim, mh, mdim, fh, fdim, fvdim, n, chunk, side, groups=1, rank=64, vocab=151936, rot=None):
        att = RotaryAttentionSpec(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, rot_dims=rot or dim,
                                  rot_base=500000.0, softcap=30.0, chunk=chunk)
        specs, source = [], None
        for i in range(n):
            if i % 3 == 0:
                mixer = TokenShiftMemorySpec(mh, mdim, rank, D)
            elif i % 3 == 1:
                mixer = ForgetGateMemorySpec(fh, fdim, fvdim)
            else:                                 # every other attention layer reads the cache of the one before it
                mixer = att if source is None else dataclasses.replace(att, kv_from=source)
                source = i if source is None else None
            specs.append(LayerSpec(mixer, ff, "xielu"))
        return cls(family="tovalix", vocab_size=vocab, embed_dim=D, layer_specs=tuple(specs), norm_groups=groups, embed_norm=True,
                   token_side=side)

    @classmethod
    def tovalix_tiny(cls) -> "StackConfig":
        return cls._tovalix(96, 160, 4, 2, 32, 3, 32, 2, 40, 24, 6, 24, 8, groups=3, rank=8, vocab=384, rot=16)

    @classmethod
    def tovalix_2b(cls) -> "StackConfig":
        return cls._tovalix(2048, 8192, 16, 8, 128, 32, 64, 16, 128, 128, 24, 1024, 64)

    @classmethod
    def tovalix_8b(cls) -> "StackConfig":
        return cls._tovalix(4096, 16384, 32, 8, 128, 64, 64, 32, 128, 128, 30, 1024, 128)


    @classmethod
    def _zikezen(cls, D, ff, heads, kv, dim, mh, mdim, mvdim, n, loop, window, experts, top, eff, side, rank=64, vocab=151936,
                 positions=16384, rot=None) -> "StackConfig":
        att = RotaryAttentionSpec(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, rot_dims=rot or dim // 2,
                                  rot_base=500000.0, window=window, interleaved=True, rot_scaling=(8.0, 1.0, 4.0, positions // 2),
                                  head_weights=True, sink=0.0, out_bias=False, fit_heads=True)
        mixer = SumSpec(att, GatedLinearSpec(mh, mdim, mvdim, 16.0, rank), 0.7, 0.6)
        specs = tuple(LayerSpec(mixer, eff, "experts", experts, top) if i % 2 else LayerSpec(mixer, ff) for i in range(n))
        return cls(family="zikezen", vocab_size=vocab, embed_dim=D, layer_specs=specs, loop=loop, token_side=side, embed_factor=2.0,
                   positions=positions, max_position=positions, loop_embed=True, post_norms=True, final_logit_softcap=30.0)

    @classmethod
    def zikezen_tiny(cls) -> "StackConfig":
        return cls._zikezen(96, 160, 4, 2, 24, 3, 16, 32, 4, (1, 3, 2), 24, 6, 2, 40, 8, rank=8, vocab=384, positions=512)

    @classmethod
    def zikezen_2b(cls) -> "StackConfig":
        return cls._zikezen(2048, 4096, 16, 8, 128, 16, 64, 128, 14, (4, 10, 2), 1024, 32, 4, 1024, 64)

    @classmethod
    def zikezen_8b(cls) -> "StackConfig":
        return cls._zikezen(4096, 8192, 32, 8, 128, 32, 64, 128, 16, (5, 11, 2), 1024, 32, 4, 2048, 128)


    @classmethod
    def _zigipel(cls, D, ff, heads, kv, dim, lheads, ldim, rot, lvdim, rank, n, loop, window, lwindow, vocab=151936, buckets=65521) -> "StackConfig":
        att = DistanceAttentionSpec(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5, window=window, keep_first=4)
        lat = LatentAttentionSpec(heads=lheads, dim=ldim, rot_dim=rot, vdim=lvdim, kv_rank=rank, scale=(ldim + rot) ** -0.5,
                                  window=lwindow, rot_dims=rot, rot_base=500000.0, rot_scaling=YarnScaling(4.0, 4096.0, 32.0, 1.0))
        specs = tuple(LayerSpec(lat if i % 2 else att, ff) for i in range(n))
        return cls(family="zigipel", vocab_size=vocab, embed_dim=D, layer_specs=specs, loop=loop, loop_input=True,
                   bigram=(buckets, 4099, 257), parallel_ff=True, token_shift=True, ff_bias=True, activation="gelu", logit_scale=0.5)

    @classmethod
    def zigipel_tiny(cls) -> "StackConfig":
        return cls._zigipel(96, 160, 4, 2, 24, 3, 16, 8, 24, 40, 4, (1, 3, 2), 24, 20, vocab=384, buckets=211)

    @classmethod
    def zigipel_2b(cls) -> "StackConfig":
        return cls._zigipel(2048, 6144, 16, 8, 128, 16, 128, 64, 128, 512, 18, (6, 12, 2), 1024, 1024)

    @classmethod
    def zigipel_8b(cls) -> "StackConfig":
        return cls._zigipel(4096, 12288, 32, 8, 128, 32, 128, 64, 128, 512, 24, (8, 14, 2), 1024, 1024)


# ------------------------------------------------------------------------------------------ config.json reader
def _parallel_spec(m: dict, shapes, prefix: str, width: int) -> ParallelSpec:
    lf, rt = m["left"], m["right"]
    mask = lf.get("mask") or {}
    rel = (shapes or {}).get(prefix + "left.rel")
    left = WindowAttentionSpec(heads=int(lf["heads"]), kv_heads=int(lf["kv_heads"]), dim=int(lf["dim"]), vdim=int(lf["vdim"]),
                               scale=float(lf["scale"]), bias_max=int(lf["bias_max"]), window=int(mask.get("size") or 0),
                               keep_first=int(mask.get("keep_first") or 0), buckets=int(rel[0]) if rel else 32)
    return ParallelSpec(left, MatrixMemorySpec(heads=int(rt["heads"]), dim=int(rt["dim"]), vdim=int(rt["vdim"]),
                                               gate_cap=float(rt["gate_cap"])))


def _rglru_spec(m: dict, shapes, prefix: str, width: int) -> RGLRUSpec:
    return RGLRUSpec(width=int(m["width"]), blocks=int(m["blocks"]), conv=int(m["conv"]))


def _rotary_spec(m: dict, shapes, prefix: str, width: int) -> RotaryAttentionSpec:
    mask, rot = m.get("mask") or {}, m.get("rot") or {}
    return RotaryAttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                               scale=float(m["scale"]), rot_dims=int(rot.get("dims") or 0), rot_base=float(rot.get("base") or 1.0),
                               softcap=float(m.get("softcap") or 0.0), chunk=int(mask.get("size") or 0),
                               kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))


def _rot_scaling(rot: dict) -> Optional[tuple]:
    s = rot.get("scaling")
    return None if not s else (float(s["factor"]), float(s["low"]), float(s["high"]), float(s["original"]))


def _sum_spec(m: dict, shapes, prefix: str, width: int) -> SumSpec:
    lf, rt = m["left"], m["right"]
    mask, rot = lf.get("mask") or {}, lf.get("rot") or {}
    left = RotaryAttentionSpec(heads=int(lf["heads"]), kv_heads=int(lf["kv_heads"]), dim=int(lf["dim"]), vdim=int(lf["vdim"]),
                               scale=float(lf["scale"]), rot_dims=int(rot.get("dims") or 0), rot_base=float(rot.get("base") or 1.0),
                               window=int(mask.get("size") or 0), interleaved=True, rot_scaling=_rot_scaling(rot), head_weights=True,
                               sink=0.0, out_bias=False, fit_heads=True)
    a1 = (shapes or {}).get(prefix + "right.a1")
    right = GatedLinearSpec(heads=int(rt["heads"]), dim=int(rt["dim"]), vdim=int(rt["vdim"]), tau=float(rt["tau"]),
                            decay_rank=int(a1[0]) if a1 else 16)
    return SumSpec(left, right, float(m["left_scale"]), float(m["right_scale"]))


def _wkv_spec(m: dict, shapes, prefix: str, width: int) -> TokenShiftMemorySpec:
    w1 = (shapes or {}).get(prefix + "w1")
    return TokenShiftMemorySpec(heads=int(m["heads"]), dim=int(m["dim"]), decay_rank=int(w1[0]) if w1 else 64, width=width)


def _hgrn2_spec(m: dict, shapes, prefix: str, width: int) -> ForgetGateMemorySpec:
    return ForgetGateMemorySpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))


def _distance_spec(m: dict, shapes, prefix: str, width: int) -> DistanceAttentionSpec:
    mask = m.get("mask") or {}
    return DistanceAttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                 scale=float(m["scale"]), window=int(mask.get("size") or 0), keep_first=int(mask.get("keep_first") or 0))


def _yarn(rot: dict) -> Optional[YarnScaling]:
    s = rot.get("scaling")
    return None if not s else YarnScaling(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"]))


def _latent_spec(m: dict, shapes, prefix: str, width: int) -> LatentAttentionSpec:
    mask, rot = m.get("mask") or {}, m["rot"]
    return LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                               kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), window=int(mask.get("size") or 0),
                               rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), rot_scaling=_yarn(rot))


@dataclass(frozen=True)
class Design:
    family: str
    mixers: dict                        # layer type in config.json -> reader of its mixer
    ff_kind: str                        # what a "dense" feed-forward is
    embed_norm: bool = False
    experts: bool = False               # layers may have a mixture of experts
    post_norms: bool = False            # a norm behind every sublayer
    loop_embed: bool = False
    options: tuple = ()                 # further fields of StackConfig that the design fixes: (name, value)


ARCHITECTURES = {
    "Roluzen": Design("roluzen", {"rglru": _rglru_spec, "parallel": _parallel_spec}, "glu"),
    "Tovalix": Design("tovalix", {"wkv": _wkv_spec, "hgrn2": _hgrn2_spec, "attention": _rotary_spec}, "xielu", embed_norm=True),
    "Zikezen": Design("zikezen", {"parallel": _sum_spec}, "glu", experts=True, post_norms=True, loop_embed=True),
    "Zigipel": Design("zigipel", {"attention": _distance_spec, "latent_attention": _latent_spec}, "glu",
                      options=(("loop_input", True), ("parallel_ff", True), ("token_shift", True), ("ff_bias", True),
                               ("activation", "gelu"))),
}
STACK_FAMILIES = tuple(d.family for d in ARCHITECTURES.values())


def is_stack_json(c: dict) -> bool:
    return c.get("architecture") in ARCHITECTURES


def describes_layer_stack(path: str) -> bool:
    """Whether the checkpoint directory `path` holds a layer-stack model's config.json."""
    try:
        with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
            return is_stack_json(json.load(f))
    except (OSError, ValueError):
        return False


def config_from_stack_json(src: Union[str, dict], dtype: Optional[torch.dtype] = None, shapes: Optional[dict] = None,
                           **overrides) -> StackConfig:
    """`src`: a checkpoint directory, a config.json path or the parsed dict. Sizes that only a tensor's shape tells (rows
    of the bias tables, the decays' bottleneck) come from the safetensors headers of the directory, or from `shapes` (name -> shape)."""
    c = src
    if isinstance(src, str):
        path = os.path.join(src, "config.json") if os.path.isdir(src) else src
        with open(path, encoding="utf-8") as f:
            c = json.load(f)
        if shapes is None:
            from .safetensors_loader import tensor_shapes
            shapes = tensor_shapes(os.path.dirname(path))
    design, width, specs = ARCHITECTURES[c["architecture"]], int(c["width"]), []
    for i, layer in enumerate(c["layers"]):
        if layer["type"] not in design.mixers:
            raise ValueError(f"layer {i}: no mixer {layer['type']!r} in this framework")
        mlp = layer.get("mlp")
        mixer = design.mixers[layer["type"]](layer["mixer"], shapes, f"l{i}.mix.", width)
        if mlp is None:
            specs.append(LayerSpec(mixer, None, design.ff_kind))
        elif mlp.get("kind") == "dense":
            specs.append(LayerSpec(mixer, int(mlp["ff"]), design.ff_kind))
        elif mlp.get("kind") == "moe" and design.experts:
            specs.append(LayerSpec(mixer, int(mlp["expert"]["ff"]), "experts", int(mlp["router"]["experts"]), int(mlp["router"]["top"])))
        else:
            raise ValueError(f"layer {i}: no feed-forward {mlp.get('kind')!r} in this framework")
    lp = c.get("loop")
    positions = int(c.get("max_positions") or 0)
    emb = c.get("embedding") or {}
    pairs = emb.get("bigram")
    kw = dict(family=design.family, vocab_size=int(c["vocab"]), embed_dim=width, norm_groups=int(c["norm"].get("groups") or 1),
              embed_norm=design.embed_norm, token_side=int((c.get("token_side") or {}).get("dim") or 0),
              norm_eps=float(c["norm"]["eps"]), layer_specs=tuple(specs),
              loop=None if not lp else (int(lp["start"]), int(lp["stop"]), int(lp["times"])),
              streams=int(c.get("streams") or 0), dtype=dtype or torch.bfloat16, post_norms=design.post_norms,
              loop_embed=design.loop_embed, embed_factor=float(emb.get("scale") or 1.0),
              final_logit_softcap=float(c.get("logit_softcap") or 0.0), positions=positions,
              bigram=None if not pairs else (int(pairs["buckets"]), int(pairs["mul_prev"]), int(pairs["mul_cur"])),
              logit_scale=1.0 if c.get("logit_scale") is None else float(c["logit_scale"]), **dict(design.options))
    if positions:
        kw["max_position"] = positions
    kw.update(overrides)
    return StackConfig(**kw)


# --------------------------------------------------------------------------------------------------- the model
class HyperConnection(nn.Module):
    """How a sublayer reads and writes the residual streams: `weight_in` [S], `weight_out` [S], `mix` [S from, S to]."""

    def __init__(self, streams: int, dtype, device=None):
        super().__init__()
        S = streams
        self.weight_in = nn.Parameter(torch.full((S,), 1.0 / S, dtype=dtype, device=device))
        self.weight_out = nn.Parameter(torch.ones(S, dtype=dtype, device=device))
        self.mix = nn.Parameter(torch.eye(S, dtype=dtype, device=device))


class PlainMLP(nn.Module):
    """down(xielu(up x)); `act` holds the activation's two numbers."""

    def __init__(self, width: int, ff: int, dtype, device=None):
        super().__init__()
        self.up_proj = Linear(width, ff, False, dtype, device)
        self.down_proj = Linear(ff, width, False, dtype, device)
        self.act = nn.Parameter(torch.full((2,), 0.5, dtype=dtype, device=device))


class ExpertsMLP(nn.Module):
    """sum_j s_j expert_j(x) over the `top` experts with the largest softmax score + correction, weighted by the score itself;
    an expert is silu-gated. Expert weights are stacked [E, F, D] (gate, up) and [E, D, F] (down)."""

    def __init__(self, width: int, ff: int, experts: int, top: int, dtype, device=None):
        super().__init__()
        self.top = top
        self.router = Linear(width, experts, False, dtype, device)
        self.correction = nn.Parameter(torch.zeros(experts, dtype=dtype, device=device))
        self.gate_proj = nn.Parameter(torch.empty(experts, ff, width, dtype=dtype, device=device))
        self.up_proj = nn.Parameter(torch.empty(experts, ff, width, dtype=dtype, device=device))
        self.down_proj = nn.Parameter(torch.empty(experts, width, ff, dtype=dtype, device=device))


class TokenSide(nn.Module):
    """A layer's token input: norm(proj(gelu(gate x) * e))."""

    def __init__(self, width: int, dim: int, eps: float, dtype, device=None):
        super().__init__()
        self.gate_proj = Linear(width, dim, False, dtype, device)
        self.proj = Linear(dim, width, False, dtype, device)
        self.norm = RMSNorm(width, eps, False, dtype, device)


class StackLayer(nn.Module):
    def __init__(self, cfg: StackConfig, spec: LayerSpec, device=None):
        super().__init__()
        D, dt, eps = cfg.embed_dim, cfg.dtype, cfg.norm_eps
        self.spec = spec
        self.input_layernorm = RMSNorm(D, eps, False, dt, device)
        self.mixer = create_mixer(spec.mixer, D, eps, dt, device)
        self.hc1 = HyperConnection(cfg.streams, dt, device) if cfg.streams else None
        self.post_attention_layernorm = self.mlp = self.hc2 = self.post_attn_norm = self.post_ffw_norm = None
        if cfg.post_norms:
            self.post_attn_norm = RMSNorm(D, eps, False, dt, device)
        # how much of the row before a mixer reads, per channel
        self.shift = nn.Parameter(torch.full((D,), 0.5, dtype=dt, device=device)) if cfg.token_shift else None
        if spec.ff is not None:
            if not cfg.parallel_ff:
                self.post_attention_layernorm = RMSNorm(D, eps, False, dt, device)
            if cfg.post_norms:
                self.post_ffw_norm = RMSNorm(D, eps, False, dt, device)
            if spec.ff_kind == "experts":
                self.mlp = ExpertsMLP(D, spec.ff, spec.experts, spec.top, dt, device)
            elif spec.ff_kind == "xielu":
                self.mlp = PlainMLP(D, spec.ff, dt, device)
            else:                       # the generic gated MLP reads only these sizes
                self.mlp = MLP(ModelConfig(embed_dim=D, hidden_dim=spec.ff, activation=cfg.activation, dtype=dt), device, cfg.ff_bias)
            self.hc2 = HyperConnection(cfg.streams, dt, device) if cfg.streams else None
        self.side = TokenSide(D, cfg.token_side, eps, dt, device) if cfg.token_side else None


class StackModel(nn.Module):
    def __init__(self, cfg: StackConfig, device=None):
        super().__init__()
        self.config = cfg
        dt = cfg.dtype
        self.embed_tokens = nn.Parameter(torch.empty(cfg.vocab_size, cfg.embed_dim, dtype=dt, device=device))
        self.embed_norm = RMSNorm(cfg.embed_dim, cfg.norm_eps, False, dt, device) if cfg.embed_norm else None
        self.pos_embed = self.side_embed = self.bigram_embed = self.loop_in = self.loop_step = None
        if cfg.bigram:              # a row per bucket of token pairs, and one for a sequence's first token
            self.bigram_embed = nn.Parameter(torch.empty(cfg.bigram[0] + 1, cfg.embed_dim, dtype=dt, device=device))
        if cfg.loop_input and cfg.loop is not None:
            self.loop_in = Linear(2 * cfg.embed_dim, cfg.embed_dim, False, dt, device)
            self.loop_step = nn.Parameter(torch.zeros(cfg.loop[2], cfg.embed_dim, dtype=dt, device=device))
        if cfg.positions:
            self.pos_embed = nn.Parameter(torch.empty(cfg.positions, cfg.embed_dim, dtype=dt, device=device))
        if cfg.token_side:          # row of a token: one part of `token_side` columns per layer
            self.side_embed = nn.Parameter(torch.empty(cfg.vocab_size, cfg.num_layers * cfg.token_side, dtype=dt, device=device))
        self.layers = nn.ModuleList([StackLayer(cfg, s, device) for s in cfg.layer_specs])
        self.norm = RMSNorm(cfg.embed_dim, cfg.norm_eps, False, dt, device)
        self.lm_head = nn.Parameter(torch.empty(cfg.vocab_size, cfg.embed_dim, dtype=dt, device=device))
        self.tp = None
        self._exec = None

    @torch.no_grad()
    def init_weights(self, seed: int = 0, std: float = 0.02) -> "StackModel":
        gen = torch.Generator(device=self.embed_tokens.device).manual_seed(seed)
        for name, p in self.named_parameters():
            if name.endswith((".mix", "_bias")):
                continue
            if p.dim() >= 2:
                p.normal_(0.0, std, generator=gen)
            elif name.endswith("bias"):
                p.zero_()
        for layer in self.layers:
            layer.mixer.init_special()
        return self

    def head_weight(self) -> torch.Tensor:
        return self.lm_head

    def compute_final_logits(self, hidden):
        z = F.lm_head_logits(hidden, self.head_weight(), softcap=self.config.final_logit_softcap)
        return z if self.config.logit_scale == 1.0 else z * self.config.logit_scale

    def token_logprobs(self, hidden, targets, *, temperature: float = 1.0, want_entropy: bool = False, chunk: Optional[int] = None):
        return F.lm_head_logprobs(hidden, self.head_weight(), targets, softcap=self.config.final_logit_softcap,
                                  temperature=temperature / self.config.logit_scale, want_entropy=want_entropy, chunk=chunk or self.config.logprob_chunk)

    @property
    def num_params(self) -> int:
        return sum(p.numel() for p in self.parameters())

    def executor(self):
        from .stack_exec import StackExecutor
        if self._exec is None:
            self._exec = StackExecutor(self)
        return self._exec

    @torch.no_grad()
    def forward(self, input_tokens, positions=None, cache=None, attention_mask=None, segment_ids=None, skip_lm_head: bool = False,
                output_hidden_states: bool = False, **unused):
        """Whole sequences [B, T] (rows may be padded: segment id 0; one segment per row) -> (logits or hidden states, None).
        Forward only; sampling goes through `generate.engine.PagedEngine`, which keeps the cache and the states."""
        if cache is not None or attention_mask is not None:
            raise NotImplementedError("layer-stack models keep their cache and state in PagedEngine: sample through it")
        from ..generate.engine import PagePool
        from ..ops.ragged import RaggedBatch
        B, T = input_tokens.shape
        dev = self.embed_tokens.device
        keep = torch.ones(B, T, dtype=torch.bool) if segment_ids is None else (segment_ids.cpu() > 0)
        if segment_ids is not None and int(segment_ids.max()) > 1:
            raise NotImplementedError("packed rows (several segments) are not scored by layer-stack models")
        toks = input_tokens.cpu()
        rows = [toks[b][keep[b]].tolist() for b in range(B)]
        if self.config.positions and max(map(len, rows), default=0) > self.config.positions:
            raise ValueError(f"rows of more than {self.config.positions} tokens: the model has no position beyond")
        pages = [-(-max(len(r), 1) // 64) for r in rows]
        pool = PagePool(self.config, sum(pages), 64, B, max(pages), dev, self.config.dtype, prefix_caching=False)
        work = []
        for b, r in enumerate(rows):
            pool.open(b, r, 0)
            if r:
                work.append((b, 0, r))
        pool.sync_table()
        ex = self.executor()
        ex.refresh()
        h = ex.forward(RaggedBatch.build(work, dev), pool)
        hidden = torch.zeros(B, T, h.shape[-1], dtype=h.dtype, device=dev)
        hidden[keep.to(dev)] = h
        return (hidden if skip_lm_head or output_hidden_states else self.compute_final_logits(hidden)), None


