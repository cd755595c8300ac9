"""Runs a `models.stack.StackModel` on ragged batches: prompts, portions of prompts and decoded tokens of any mix go
through the same function, reading and writing the engine's paged cache and slot states.

Between two sublayers one kernel closes the one before (hyper-connection write) and opens the one after (hyper-connection
read and norm). Projections that share an input run as one GEMM over weights joined in memory; where mixer and feed-forward
run side by side, the heads and the gated activation land in one row, which one GEMM takes back. bf16 models run on the
package's tcgen05 GEMMs, with fp32 accumulation; 32-bit models use library GEMMs in full precision (no TF32)."""
from __future__ import annotations

import math
from typing import Callable, Optional

import torch

from ..ops import kernels as K
from ..ops import stack_kernels as SK
from ..ops.ragged import RaggedBatch
from .mixers import (TILE_HEADS, DistanceAttention, ForgetGateMemory, GatedLinearAttention, LatentAttention, ParallelMixer, RGLRUMixer,
                     RotaryAttention, SumMixer, TokenShiftMemory, YarnScaling)
from .stack import ExpertsMLP, PlainMLP


def _plain(mods) -> None:
    if any(m.quant is not None or (m.lora_a is not None and m.lora_enabled) for m in mods):
        raise NotImplementedError("layer-stack models run without adapters or quantised weights")


def joint_weight(mods):
    """One [sum(out_i), in] tensor over the weights of `mods` (moved there once; the modules keep views), and the joint
    bias (zeros for modules without one) or None. Adapters and quantised bases are not supported on these models."""
    _plain(mods)
    ws = [m.weight for m in mods]
    rows, base = sum(w.shape[0] for w in ws), ws[0].data
    off, adjacent = base.storage_offset(), True
    for w in ws:
        if w.untyped_storage().data_ptr() != base.untyped_storage().data_ptr() or w.storage_offset() != off or not w.is_contiguous():
            adjacent = False
            break
        off += w.numel()
    if adjacent:
        joint = base.as_strided((rows, base.shape[1]), (base.shape[1], 1), base.storage_offset())
    else:
        joint = torch.cat([w.data for w in ws], 0)
        r = 0
        for w in ws:
            w.data = joint[r:r + w.shape[0]]
            r += w.shape[0]
    bias = None
    if any(m.bias is not None for m in mods):
        bias = torch.cat([m.weight.new_zeros(m.weight.shape[0]) if m.bias is None else m.bias.data for m in mods])
    return joint, bias


def side_by_side(params, dim: int) -> torch.Tensor:
    """The parameters joined along `dim` in one contiguous tensor (moved there once; they stay views of it)."""
    sizes = [p.shape[dim] for p in params]
    shape = list(params[0].shape)
    shape[dim] = sum(sizes)
    base, off = params[0].data, 0
    stride = [1] * len(shape)
    for i in range(len(shape) - 2, -1, -1):
        stride[i] = stride[i + 1] * shape[i + 1]
    for p, n in zip(params, sizes):
        if p.data.untyped_storage().data_ptr() != base.untyped_storage().data_ptr() or list(p.stride()) != stride or \
                p.storage_offset() != base.storage_offset() + off * stride[dim]:
            break
        off += n
    else:
        return base.as_strided(shape, stride, base.storage_offset())
    joint = torch.cat([p.data for p in params], dim)
    for p, part in zip(params, joint.split(sizes, dim)):
        p.data = part
    return joint


def linear(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, out_dtype: Optional[torch.dtype] = None,
           packed=None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x @ w^T (+ bias), fp32 accumulation, output in `out_dtype` (default: x's) or in `out`, which may be columns of wider rows."""
    out_dtype = out_dtype or (x.dtype if out is None else out.dtype)
    if x.dtype == torch.bfloat16:
        if packed is not None:
            return K.gemm_packed(x, packed, bias=bias, out_dtype=out_dtype, out=out)
        if x.shape[1] % 8 == 0:
            if x.stride(0) % 8 or x.data_ptr() % 16:        # columns of a wider row that TMA cannot address
                x = x.contiguous()
            return K.gemm(x, w, bias=bias, out_dtype=out_dtype, out=out)
    if out is not None:
        return out.copy_(linear(x, w, bias, out_dtype))
    prev = torch.backends.cuda.matmul.allow_tf32
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        if x.dtype != out_dtype:
            x, w, bias = x.to(out_dtype), w.to(out_dtype), None if bias is None else bias.to(out_dtype)
        return torch.nn.functional.linear(x, w, bias)
    finally:
        torch.backends.cuda.matmul.allow_tf32 = prev


def _per_head(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x [n, heads, K] with a matrix per head w [heads, K, N] -> [n, heads, N], by the library in full precision."""
    prev = torch.backends.cuda.matmul.allow_tf32
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        return torch.bmm(x.transpose(0, 1), w).transpose(0, 1)
    finally:
        torch.backends.cuda.matmul.allow_tf32 = prev


FEW_OUTPUTS = 512       # in a decode step, products with at most this many outputs split the contraction inside a CTA


def rope_frequencies(dims: int, base: float, scaling: Optional[tuple] = None, device=None) -> torch.Tensor:
    """fp64 [dims / 2]: base^(-2 i / dims). `scaling` = (factor, low, high, original context), as Llama 3.1 has it: frequencies
    that turn fewer than `low` times over the original context are divided by the factor, those that turn more than `high` times
    stay, in between the two are mixed linearly in the number of turns. With a `YarnScaling` the mix is linear in the number of the
    pair, between the (rounded) pairs that turn `fast` and `slow` times."""
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64, device=device) / max(dims, 1))
    if scaling is None or not dims:
        return f
    if isinstance(scaling, YarnScaling):
        pair = lambda turns: dims * math.log(scaling.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))  # noqa: E731
        lo, hi = max(math.floor(pair(scaling.fast)), 0), min(math.ceil(pair(scaling.slow)), dims - 1)
        far = ((torch.arange(dims // 2, dtype=torch.float64, device=device) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / scaling.factor * far + f * (1.0 - far)
    factor, low, high, original = scaling
    turns = original * f / (2.0 * math.pi)
    keep = ((turns - low) / (high - low)).clamp(0.0, 1.0) if high > low else (turns >= low).to(f.dtype)
    return torch.where(turns > high, f, torch.where(turns < low, f / factor, (1.0 - keep) * f / factor + keep * f))


def rope_table(positions: int, dims: int, base: float, device, scaling: Optional[tuple] = None) -> tuple:
    """cos / sin fp32 [positions, dims / 2] of the angles position * frequency, from fp64 (times a `YarnScaling`'s size)."""
    f = rope_frequencies(dims, base, scaling, device)
    a = torch.arange(positions, dtype=torch.float64, device=device)[:, None] * f
    size = scaling.size if isinstance(scaling, YarnScaling) else 1.0
    return (size * a.cos()).float(), (size * a.sin()).float()


class StackExecutor:
    def __init__(self, model):
        self.model = model
        self.cfg = model.config
        self.runs = self.cfg.runs()
        self.kv_src = self.cfg.kv_sources()
        self._mix = {RGLRUMixer: self._rglru, ParallelMixer: self._parallel, RotaryAttention: self._rotary,
                     TokenShiftMemory: self._shift_memory, ForgetGateMemory: self._forget_memory,
                     GatedLinearAttention: self._gated_linear, SumMixer: self._sum}
        # mixers whose heads can land in columns of a wider row, before their output projection
        self._heads = {DistanceAttention: self._distance_heads, LatentAttention: self._latent_heads}
        self.restarts = self.cfg.restarts() if self.cfg.loop_embed else set()
        self.starts = self.cfg.loop_starts() if self.cfg.loop_input else {}
        self._rope: dict = {}       # kept for good: captured decode graphs point at the tables
        self._far: dict = {}        # (layer, positions) -> distance bias, kept likewise
        self.dtype = model.embed_tokens.dtype
        self.pk: Callable = lambda i, name: None        # packed decode weights, set by the engine
        self.plain = False          # bf16 through the simple kernels of the 32-bit path (a cross-check, slow)
        self._one = None
        self.w: list = []
        self.refresh()

    # ------------------------------------------------------------------------------------------------ weights
    @torch.no_grad()
    def refresh(self) -> None:
        """(Re)build everything derived from the parameters. Buffers keep their addresses, so that a captured decode
        graph stays valid after an in-place weight update."""
        fresh = []
        for layer in self.model.layers:
            d = {}
            for name, mods in zip(("proj", "gates"), layer.mixer.fused_groups()):
                d[name], d[name + "_bias"] = joint_weight(mods)
            if isinstance(layer.mixer, ParallelMixer):
                d["bias"] = layer.mixer.left.bias_table()
                d["gates_bias"] = None                   # added by the recurrence in fp32
            if isinstance(layer.mixer, ForgetGateMemory):
                d["gates_bias"] = None
            if isinstance(layer.mixer, TokenShiftMemory):
                d["mu"] = layer.mixer.mu()
            if isinstance(layer.mixer, SumMixer):
                outs = [layer.mixer.left.o_proj, layer.mixer.right.o_proj]
                _plain(outs)
                d["o"] = side_by_side([m.weight for m in outs], 1)
            if self.cfg.parallel_ff:
                outs = [layer.mixer.o_proj] + ([] if layer.mlp is None else [layer.mlp.down_proj])
                _plain(outs)
                d["o"] = side_by_side([m.weight for m in outs], 1)
                d["o_bias"] = None if layer.mlp is None or layer.mlp.down_proj.bias is None else layer.mlp.down_proj.bias.data
            if isinstance(layer.mixer, (DistanceAttention, LatentAttention)):
                d["sinks"] = layer.mixer.sink.detach().float()
            if isinstance(layer.mixer, LatentAttention):
                sp, w = layer.mixer.spec, layer.mixer.uk_proj.weight
                _plain([layer.mixer.uk_proj, layer.mixer.uv_proj])
                if sp.tiled(w.dtype):
                    d["expand"] = layer.mixer.expansion(sp.stored(w.dtype)[0])
            if isinstance(layer.mlp, PlainMLP):
                d["up"], _ = joint_weight([layer.mlp.up_proj])
            elif isinstance(layer.mlp, ExpertsMLP):
                _plain([layer.mlp.router])
                d["experts_gu"] = side_by_side([layer.mlp.gate_proj, layer.mlp.up_proj], 1)
            elif layer.mlp is not None:
                d["gu"], d["gu_bias"] = joint_weight([layer.mlp.gate_proj, layer.mlp.up_proj])
            fresh.append(d)
        for (i, positions), table in self._far.items():
            table.copy_(self.model.layers[i].mixer.bias_table(positions))
        for new, old in zip(fresh, self.w):
            for k, v in old.items():
                if v is not None and v.shape == new[k].shape:
                    if v.data_ptr() != new[k].data_ptr():
                        v.copy_(new[k])
                    new[k] = v
        self.w = fresh

    def pack_sources(self) -> list:
        """Per layer, the weights the engine may keep in packed form for decoding (`PagedEngine._pack_all`)."""
        out = []
        for layer, d in zip(self.model.layers, self.w):
            src = {k: d[k] for k in ("proj", "gates", "gu", "up", "o") if k in d}
            if layer.mlp is not None and not isinstance(layer.mlp, ExpertsMLP) and not self.cfg.parallel_ff:
                src["down"] = layer.mlp.down_proj.weight.data
            out.append(src)
        return out

    def _hc(self, hc):
        if hc is not None:
            return hc.weight_in, hc.weight_out, hc.mix
        if self._one is None:
            self._one = torch.ones(1, dtype=self.dtype, device=self.model.embed_tokens.device)
        return self._one, self._one, self._one

    # ------------------------------------------------------------------------------------------------ sublayers
    def _rglru(self, i, m: RGLRUMixer, h, rb: RaggedBatch, pool, r):
        d = self.w[i]
        proj = linear(h, d["proj"], d["proj_bias"], packed=self.pk(i, "proj") if rb.decode else None)
        o = SK.rglru(proj, m.spec.width, 0, m, rb, pool.state[r], self.plain)
        return (linear(o, m.o_proj.weight), None, None, None)

    def _parallel(self, i, m: ParallelMixer, h, rb: RaggedBatch, pool, r):
        d, lf, rt = self.w[i], m.left, m.right
        a, s = lf.spec, rt.spec
        proj = linear(h, d["proj"], packed=self.pk(i, "proj") if rb.decode else None)
        if rb.decode and h.dtype == torch.bfloat16 and h.shape[1] % 8 == 0:
            gates = SK.few_outputs(h, d["gates"])
        else:
            gates = linear(h, d["gates"], out_dtype=torch.float32)
        off, cols = [], 0
        for width in (a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim, a.heads * a.vdim, s.heads * s.dim, s.heads * s.dim,
                      s.heads * s.vdim, s.heads * s.vdim):
            off.append(cols)
            cols += width
        q = SK.qk_norm_write(proj, off[0], off[1], off[2], lf.q_norm.weight, lf.k_norm.weight, lf.eps, rb, pool.table,
                             pool.page_size, pool.k[r], pool.v[r], a.heads * a.dim)
        att = self._attend(q, a, d["bias"], rb, pool, r)
        o = SK.mlstm(proj, off[4], off[5], off[6], gates, rt.i_proj.bias, rt.f_proj.bias, s.gate_cap, rb, s.heads, s.dim, s.vdim,
                     pool.state[r], self.plain)
        a1, a2 = SK.gate_outputs(att, o, proj, off[3], off[7], rt.norm.weight, rt.eps, s.heads, s.vdim)
        return (linear(a1, lf.o_proj.weight), linear(a2, rt.o_proj.weight), m.left_norm.weight, m.right_norm.weight)

    def _rotary(self, i, m: RotaryAttention, h, rb: RaggedBatch, pool, r):
        d = self.w[i]
        proj = linear(h, d["proj"], d["proj_bias"], packed=self.pk(i, "proj") if rb.decode else None)
        att = self._rotary_heads(m, proj, rb, pool, r)
        return (linear(att, m.o_proj.weight, m.o_proj.bias), None, None, None)

    def _rotary_heads(self, m: RotaryAttention, proj, rb: RaggedBatch, pool, r, **kw):
        """Attention of the projected rows (queries, keys and values in their first columns), before the output projection."""
        a, src = m.spec, self.kv_src[r]
        cos, sin = self._rope_tables(a, pool, proj.device)
        nq, kv = a.heads * a.dim, 0 if a.kv_from is not None else a.kv_heads
        q = SK.rope_norm_write(proj, 0, nq, nq + kv * a.dim, cos, sin, a.rot_dims, m.eps, rb, pool.table, pool.page_size, a.heads,
                               kv, a.dim, a.vdim, pool.k[src], pool.v[src], q_w=None if m.q_norm is None else m.q_norm.weight,
                               k_w=None if m.k_norm is None else m.k_norm.weight, interleaved=a.interleaved,
                               stored=a.stored(proj.dtype))
        return self._attend(q, a, None, rb, pool, src, **kw)

    def _rope_tables(self, a, pool, device) -> tuple:
        key = (a.rot_dims, a.rot_base, a.rot_scaling, pool.max_pages * pool.page_size)
        if key not in self._rope:
            self._rope[key] = rope_table(key[3], a.rot_dims, a.rot_base, device, a.rot_scaling)
        return self._rope[key]

    def _distance_heads(self, i, m: DistanceAttention, h, rb: RaggedBatch, pool, r, out) -> None:
        d, a = self.w[i], m.spec
        nq, nk, nv = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
        cols = nq + nk + nv + a.heads
        row = torch.empty((h.shape[0], -(-cols // 8) * 8), dtype=h.dtype, device=h.device)
        proj = linear(h, d["proj"], d["proj_bias"], packed=self.pk(i, "proj") if rb.decode else None, out=row[:, :cols])
        wide, wide_v = a.stored(h.dtype)
        # queries stay where they are: what a wider head reads behind its own columns meets the zeros behind the stored key
        here = a.dim % 8 == 0 and (a.heads - 1) * a.dim + wide <= row.shape[1]
        q = SK.rope_norm_write(proj, 0, nq, nq + nk, None, None, 0, m.eps, rb, pool.table, pool.page_size, 0 if here else a.heads,
                               a.kv_heads, a.dim, a.vdim, pool.k[r], pool.v[r], stored=(wide, wide_v), norm_qk=False, norm_v=True)
        if here:
            q = row.as_strided((row.shape[0], a.heads, wide), (row.stride(0), a.dim, 1))
        self._attend(q, a, self._distance_bias(i, m, pool), rb, pool, r, out=out, sinks=d["sinks"], gate=proj[:, nq + nk + nv:])

    def _distance_bias(self, i, m: DistanceAttention, pool) -> torch.Tensor:
        key = (i, pool.max_pages * pool.page_size)
        if key not in self._far:
            self._far[key] = m.bias_table(key[1])
        return self._far[key]

    def _latent_heads(self, i, m: LatentAttention, h, rb: RaggedBatch, pool, r, out) -> None:
        """Portions of prompts expand the latents of their window to keys and values for the flash attention; single tokens and
        short portions attend in the absorbed form, as everything does in the general kernel."""
        d, sp, n = self.w[i], m.spec, h.shape[0]
        H, qd, R, lat = sp.heads, sp.dim + sp.rot_dim, sp.kv_rank, pool.k[r]
        proj = linear(h, d["proj"], d["proj_bias"], packed=self.pk(i, "proj") if rb.decode else None)
        SK.latent_write(proj, H * qd, m.kv_norm.weight, *self._rope_tables(sp, pool, h.device), sp.rot_dims, m.eps, rb, pool.table,
                        pool.page_size, H, sp.dim, sp.rot_dim, R, lat)
        q, W = proj[:, :H * qd].unflatten(1, (H, qd)), lat.shape[-1]
        uk, uv = m.uk_proj.weight.data.view(H, sp.dim, R), m.uv_proj.weight.data.view(H, sp.vdim, R)
        if self.plain or not sp.tiled(h.dtype) or pool.page_size % 64:
            full = q.new_zeros((n, H, W))
            full[:, :, :R] = _per_head(q[:, :, :sp.dim], uk)
            full[:, :, R:R + sp.rot_dim] = q[:, :, sp.dim:]
            att = SK.window_attn(full, lat, lat, rb, pool.table, pool.page_size, sp, None, sinks=d["sinks"], sizes=(1, sp.width, R, W, W))
            out.unflatten(1, (H, sp.vdim)).copy_(_per_head(att.view(n, H, R), uv.transpose(1, 2)))
            return
        to = out if out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0 else torch.empty(out.shape, dtype=out.dtype, device=out.device)
        plan = rb.latent_plan(sp.window)
        if plan.blocks is not None:
            wide, wide_v = sp.tile_heads()
            rows = SK.latent_gather(lat, *plan.blocks, pool.table, pool.page_size)
            kv = linear(rows[:, :d["expand"].shape[1]], d["expand"])
            keys = H * (sp.dim if sp.split_keys else wide)
            qw = proj.as_strided((n, H, wide), (proj.stride(0), qd, 1)) if (H - 1) * qd + wide <= proj.shape[1] else \
                torch.nn.functional.pad(q, (0, wide - qd))
            K.attn_fwd_paged(qw, kv[:, :keys], kv[:, keys:], rb, plan.table, 64, num_heads=H, num_kv_heads=H, head_dim=wide,
                             scale=sp.scale, window=sp.window, sinks=d["sinks"], out=to, value_dim=sp.vdim, tiles=plan.tiles,
                             slots=plan.entries, shared_keys=(rows, R) if sp.split_keys else None)
        count = n if plan.rows is None else plan.rows.shape[0]
        if count:
            q1 = SK.head_product(q, uk, torch.empty((count, H, W), dtype=h.dtype, device=h.device), x_rows=plan.rows, rows=count,
                                 tail=sp.rot_dim)
            att = SK.latent_decode(q1, lat, pool.table, pool.page_size, plan.slots, self._lens if plan.lens is None else plan.lens, rank=R,
                                   scale=sp.scale, window=sp.window, sinks=d["sinks"], max_ctx=pool.max_pages * pool.page_size)
            SK.head_product(att, uv, to.unflatten(1, (H, sp.vdim)), transposed=True, out_rows=plan.rows, rows=count)
        if to is not out:
            out.copy_(to)

    def _shift_memory(self, i, m: TokenShiftMemory, h, rb: RaggedBatch, pool, r):
        """h: the mixes [5, n, D] in a decode step (made by the launch before), else the normed rows."""
        sp, st = m.spec, pool.state[r]
        mixes = h if rb.decode else SK.token_shift(h, self.w[i]["mu"], st["last"], rb)
        q, k, v, g = (linear(x, p.weight) for x, p in zip(mixes, (m.r_proj, m.k_proj, m.v_proj, m.g_proj)))
        z = linear(self._few(mixes[4], m.w1_proj.weight, rb, SK.ACT_TANH), m.w2_proj.weight, out_dtype=torch.float32)
        o = SK.gated_linear(SK.GATES_BONUS, q, k, v, z, m.w0, m.u, rb, sp.heads, sp.dim, sp.dim, st["S"], m.norm.weight, m.eps, gate=g,
                            per_head=True, carry=st["last"], h=None if rb.decode else h, plain=self.plain)
        return (linear(o, m.o_proj.weight), None, None, None)

    def _forget_memory(self, i, m: ForgetGateMemory, h, rb: RaggedBatch, pool, r):
        d, sp = self.w[i], m.spec
        proj = linear(h, d["proj"], packed=self.pk(i, "proj") if rb.decode else None)
        z = linear(h, d["gates"], out_dtype=torch.float32, packed=self.pk(i, "gates") if rb.decode else None)
        nq = sp.heads * sp.dim
        o = SK.gated_linear(SK.GATES_LOWER, proj[:, :nq], None, proj[:, nq:], z, m.f_proj.bias, m.lower, rb, sp.heads, sp.dim, sp.vdim,
                            pool.state[r]["S"], m.norm.weight, m.eps, plain=self.plain)
        return (linear(o, m.o_proj.weight), None, None, None)

    def _gated_linear(self, i, m: GatedLinearAttention, h, rb: RaggedBatch, pool, r):
        proj = linear(h, self.w[i]["proj"], packed=self.pk(i, "proj") if rb.decode else None)
        return (linear(self._gated_heads(m, proj, rb, pool, r), m.o_proj.weight), None, None, None)

    def _gated_heads(self, m: GatedLinearAttention, proj, rb: RaggedBatch, pool, r, **kw):
        """The memory's read-outs, normed and gated, from the projected rows (q, k, v, gate, bottleneck)."""
        sp = m.spec
        nk, nv = sp.heads * sp.dim, sp.heads * sp.vdim
        q, k, v, g, x = proj.split([nk, nk, nv, nv, sp.decay_rank], 1)
        low = (x, m.a2_proj.weight)
        z = None if rb.decode and not self.plain and sp.vdim <= SK.STEP_WIDTH else linear(x, m.a2_proj.weight, out_dtype=torch.float32)
        return SK.gated_linear(SK.GATES_ROOT, q, k, v, z, m.a2_proj.bias, None, rb, sp.heads, sp.dim, sp.vdim, pool.state[r]["S"],
                               m.norm.weight, m.eps, gate=g, plain=self.plain, low_rank=low, q_scale=sp.dim ** -0.5, tau=sp.tau, **kw)

    def _sum(self, i, m: SumMixer, h, rb: RaggedBatch, pool, r):
        """Both mixers' heads land, scaled, in one row, which a single product takes to the residual's width."""
        d, sp = self.w[i], m.spec
        a, s = sp.left, sp.right
        proj = linear(h, d["proj"], d["proj_bias"], packed=self.pk(i, "proj") if rb.decode else None)
        na, ns = a.heads * a.vdim, s.heads * s.vdim
        o = torch.empty((h.shape[0], na + ns), dtype=h.dtype, device=h.device)
        left = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim)
        self._rotary_heads(m.left, proj, rb, pool, r, out=o[:, :na], out_scale=sp.left_scale)
        self._gated_heads(m.right, proj[:, left:], rb, pool, r, out=o[:, na:], out_scale=sp.right_scale)
        return (linear(o, d["o"], packed=self.pk(i, "o") if rb.decode else None), None, None, None)

    def _few(self, x, w, rb: RaggedBatch, act: int, **rows) -> torch.Tensor:
        """act(x w^T) for narrow w."""
        if rb.decode and x.dtype == torch.bfloat16 and x.shape[1] % 8 == 0 and w.shape[0] <= FEW_OUTPUTS:
            return SK.few_outputs(x, w, act, **rows)
        return SK.small_act(linear(x, w, out_dtype=torch.float32), x.dtype, act, **rows)

    def _side(self, i, side, x, rb: RaggedBatch):
        dim = self.cfg.token_side
        y = self._few(x, side.gate_proj.weight, rb, SK.ACT_GELU_ROW, tokens=rb.tokens, rows=self.model.side_embed, col=i * dim)
        return (linear(y, side.proj.weight), None, side.norm.weight, None)

    def _attend(self, q, a, bias, rb: RaggedBatch, pool, r, out=None, out_scale: float = 1.0, sinks=None, gate=None):
        """Tensor-core kernels where the stored heads fit them (the framework's paged decode and flash attention, extended by the
        bias, the kept tokens, the sink and the heads' gates); otherwise, and in 32-bit, the general kernel. q: [n, heads * stored], or a
        view [n, heads, stored]. `out`: columns that take the result."""
        wide, wide_v = a.stored(q.dtype)
        fits = q.dtype == torch.bfloat16 and wide == wide_v and wide in TILE_HEADS and not self.plain and a.vdim % 8 == 0 and \
            (out is None or (out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0))
        kw = dict(scale=a.scale, softcap=a.softcap, window=a.window, chunk=a.chunk, keep_first=a.keep_first, sink=a.sink, bias=bias,
                  value_dim=a.vdim, out=out, out_scale=out_scale, sinks=sinks, gate=gate)
        fits = fits and q.stride(0) % 8 == 0 and (q.dim() == 2 or q.stride(1) % 8 == 0)
        if fits and rb.decode and a.heads // a.kv_heads <= 16:
            max_ctx = pool.table.shape[1] * pool.page_size
            span = min((s for s in (a.window, a.chunk) if s > 0), default=0)       # most keys a query sees besides the kept ones
            split = K.decode_split_tokens(rb.n, a.kv_heads, min(max_ctx, span + a.keep_first + 128) if span else max_ctx)
            return K.paged_decode(q if q.dim() == 3 else q.view(rb.n, a.heads, wide), pool.k[r], pool.v[r], pool.table, rb.slot, self._lens,
                                  num_kv_heads=a.kv_heads, page_size=pool.page_size, max_ctx=max_ctx, split_tokens=split,
                                  **kw).flatten(1)
        if fits and not rb.decode and pool.page_size % 64 == 0:
            return K.attn_fwd_paged(q, pool.k[r], pool.v[r], rb, pool.table, pool.page_size, num_heads=a.heads,
                                    num_kv_heads=a.kv_heads, head_dim=wide, **kw)
        return SK.window_attn(q, pool.k[r], pool.v[r], rb, pool.table, pool.page_size, a, bias, out=out, out_scale=out_scale,
                              sinks=sinks, gate=gate)

    def _side_by_side(self, i, layer, h, mixed, rb: RaggedBatch, pool, r):
        """Mixer (on its own input `mixed`) and feed-forward of one norm: one row takes the heads and the gated activation."""
        m, ff = layer.mixer, layer.spec.ff or 0
        heads = m.spec.heads * m.spec.vdim
        row = torch.empty((mixed.shape[0], heads + ff), dtype=mixed.dtype, device=mixed.device)
        self._heads[type(m)](i, m, mixed, rb, pool, r, row[:, :heads])
        if ff:
            self._gated(i, h, rb, row[:, heads:])
        return (linear(row, self.w[i]["o"], self.w[i]["o_bias"], packed=self.pk(i, "o") if rb.decode else None), None, None, None)

    def _gated(self, i, h, rb: RaggedBatch, out=None) -> torch.Tensor:
        """The gated activation of a feed-forward; `out`: columns of wider rows."""
        d, kind = self.w[i], K.GLU_SILU if self.cfg.activation == "silu" else K.GLU_GELU
        F = d["gu"].shape[0] // 2
        pgu = self.pk(i, "gu") if rb.decode else None
        aligned = out is None or (out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0)
        if pgu is not None and pgu.glu:
            act = K.gemm_packed(h, pgu, glu=kind, bias=d["gu_bias"], out=out if aligned else None)
            return act if out is None or aligned else out.copy_(act)
        gu = linear(h, d["gu"], d["gu_bias"], packed=pgu)
        if gu.dtype == torch.bfloat16 and F % 8 == 0 and aligned:
            return K.glu_fwd(gu[:, :F], gu[:, F:], kind, out)
        return SK.glu(gu, kind, out)

    def _mlp(self, i, mlp, h, rb: RaggedBatch):
        if isinstance(mlp, PlainMLP):
            pup = self.pk(i, "up") if rb.decode else None
            act = K.gemm_packed(h, pup, xielu=mlp.act) if pup is not None else SK.xielu_(linear(h, self.w[i]["up"]), mlp.act)
            return linear(act, mlp.down_proj.weight, packed=self.pk(i, "down") if rb.decode else None)
        if isinstance(mlp, ExpertsMLP):
            return SK.moe(h, self._router(h, mlp.router.weight, rb), mlp.correction, self.w[i]["experts_gu"], mlp.down_proj, mlp.top, rb)
        return linear(self._gated(i, h, rb), mlp.down_proj.weight, mlp.down_proj.bias, packed=self.pk(i, "down") if rb.decode else None)

    def _router(self, h, w, rb: RaggedBatch) -> torch.Tensor:
        """fp32 router logits."""
        if h.dtype == torch.bfloat16 and h.shape[1] % 8 == 0 and (rb.n <= SK.ROWS_TOKENS and w.shape[0] <= FEW_OUTPUTS):
            return SK.few_outputs(h, w)
        return linear(h, w, out_dtype=torch.float32)

    # ------------------------------------------------------------------------------------------------ the stack
    @torch.no_grad()
    def forward(self, rb: RaggedBatch, pool, layer_sums: Optional[list] = None) -> torch.Tensor:
        """Final normed hidden rows [n, D] of the batch's tokens. `pool`: the engine's PagePool (cache, page table, states).
        `layer_sums` (a list) receives the sum of the streams after every layer pass."""
        cfg, model = self.cfg, self.model
        eps, n = cfg.norm_eps, rb.n
        x = torch.empty((n, max(cfg.streams, 1), cfg.embed_dim), dtype=torch.float32, device=rb.tokens.device)
        start = dict(tokens=rb.tokens, embed=model.embed_tokens, embed_w=None if model.embed_norm is None else model.embed_norm.weight,
                     embed_scale=cfg.embed_factor, pos=model.pos_embed)
        if cfg.bigram:
            start["pairs"] = (model.bigram_embed, cfg.bigram, pool.state.tokens["last"])
        close = start                                                  # what the next stream_step closes
        pair = None                                                    # [n, 2 D]: residual and embedding output, as a pass begins
        if self.starts:
            pair = torch.empty((n, 2 * cfg.embed_dim), dtype=self.dtype, device=x.device)
            close = dict(start, start_out=pair[:, cfg.embed_dim:])

        def pending(out, hc, norm=None):
            y, y2, wy, wy2 = out
            if norm is not None:
                wy = norm.weight
            _, w_out, mix = self._hc(hc)
            return dict(y=y, y2=y2, wy=wy, wy2=wy2, mix=mix, w_out=w_out)

        if rb.decode:
            self._lens = rb.pos0 + 1                                   # keys each query sees (0: idle slot)
        ended = False                                                  # the pending sublayer ends a layer pass
        def step(w_in, norm_w, **kw):
            nonlocal ended
            total = None
            if layer_sums is not None and ended:
                total = torch.empty((n, cfg.embed_dim), dtype=torch.float32, device=x.device)
                layer_sums.append(total)
            ended = False
            return SK.stream_step(x, eps, groups=cfg.norm_groups, w_in=w_in, norm_w=norm_w, sum_out=total, rb=rb, **close, **kw)

        for r, i in enumerate(self.runs):
            layer = model.layers[i]
            if r in self.starts:
                step(None, None, raw=True, out=pair[:, :cfg.embed_dim])
                linear(pair, model.loop_in.weight, model.loop_step[self.starts[r]], out=x.view(n, -1))
                close = {}
            if cfg.parallel_ff:
                before = pool.state[r]["before"]
                if rb.decode:
                    h, mixed = step(self._hc(None)[0], layer.input_layernorm.weight, shift=(layer.shift[None], before), both=True)
                else:
                    h = step(self._hc(None)[0], layer.input_layernorm.weight)
                    mixed = SK.token_shift(h, layer.shift[None], before, rb)
                    SK.keep_last(h, before, rb)
                close = pending(self._side_by_side(i, layer, h, mixed[0], rb, pool, r), None)
                ended = True
                continue
            shifts = rb.decode and isinstance(layer.mixer, TokenShiftMemory)
            if r in self.restarts:
                close = dict(close, **start)
            h = step(self._hc(layer.hc1)[0], layer.input_layernorm.weight,
                     **(dict(shift=(self.w[i]["mu"], pool.state[r]["last"])) if shifts else {}))
            close = pending(self._mix[type(layer.mixer)](i, layer.mixer, h, rb, pool, r), layer.hc1, layer.post_attn_norm)
            if layer.mlp is not None:
                h = step(self._hc(layer.hc2)[0], layer.post_attention_layernorm.weight)
                close = pending((self._mlp(i, layer.mlp, h, rb), None, None, None), layer.hc2, layer.post_ffw_norm)
            if layer.side is not None:
                close = pending(self._side(i, layer.side, step(None, None, raw=True), rb), None)
            ended = True
        return step(None, model.norm.weight, **({"keep": pool.state.tokens["last"]} if cfg.bigram else {}))

    def logits(self, hidden: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """fp32 logits of normed hidden rows."""
        packed, scale = self.pk(len(self.model.layers), "head"), self.cfg.logit_scale
        if hidden.dtype == torch.bfloat16 and packed is not None:
            return K.gemm_packed(hidden, packed, out=out, out_dtype=torch.float32, alpha=scale)
        if hidden.dtype == torch.bfloat16 and hidden.shape[1] % 8 == 0:
            return K.gemm(hidden, self.model.head_weight(), out=out, out_dtype=torch.float32, alpha=scale)
        z = linear(hidden, self.model.head_weight(), out_dtype=torch.float32)
        z = z if scale == 1.0 else z.mul_(scale)
        return z if out is None else out.copy_(z)
