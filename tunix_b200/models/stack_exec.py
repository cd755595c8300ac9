"""Runs a `models.stack.StackModel` on ragged batches: prompts, portions of prompts and decoded tokens of any mix go
through the same function, reading and writing the engine's paged cache and slot states.

Between two sublayers one kernel closes the one before (hyper-connection write) and opens the one after (hyper-connection
read and norm). Projections that share an input run as one GEMM over weights joined in memory. bf16 models run on the
package's tcgen05 GEMMs, with fp32 accumulation; 32-bit models use library GEMMs in full precision (no TF32)."""
from __future__ import annotations

from typing import Callable, Optional

import torch

from ..ops import kernels as K
from ..ops import stack_kernels as SK
from ..ops.ragged import RaggedBatch
from .mixers import ForgetGateMemory, ParallelMixer, RGLRUMixer, RotaryAttention, TokenShiftMemory
from .stack import PlainMLP


def joint_weight(mods):
    """One [sum(out_i), in] tensor over the weights of `mods` (moved there once; the modules keep views), and the joint
    bias or None. Adapters and quantised bases are not supported on these models."""
    if any(m.quant is not None or (m.lora_a is not None and m.lora_enabled) for m in mods):
        raise NotImplementedError("layer-stack models run without adapters or quantised weights")
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
    bias = torch.cat([m.bias.data for m in mods]) if mods[0].bias is not None else None
    return joint, bias


def linear(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, out_dtype: Optional[torch.dtype] = None,
           packed=None) -> torch.Tensor:
    """x @ w^T (+ bias), fp32 accumulation, output in `out_dtype` (default: x's)."""
    out_dtype = out_dtype or x.dtype
    if x.dtype == torch.bfloat16:
        if packed is not None:
            return K.gemm_packed(x, packed, bias=bias, out_dtype=out_dtype)
        if x.shape[1] % 8 == 0:
            return K.gemm(x, w, bias=bias, out_dtype=out_dtype)
    prev = torch.backends.cuda.matmul.allow_tf32
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        if x.dtype != out_dtype:
            x, w, bias = x.to(out_dtype), w.to(out_dtype), None if bias is None else bias.to(out_dtype)
        return torch.nn.functional.linear(x, w, bias)
    finally:
        torch.backends.cuda.matmul.allow_tf32 = prev


FEW_OUTPUTS = 512       # in a decode step, products with at most this many outputs split the contraction inside a CTA


def rope_table(positions: int, dims: int, base: float, device) -> tuple:
    """cos / sin fp32 [positions, dims / 2] of the angles position * base^(-2 i / dims), from fp64."""
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64, device=device) / max(dims, 1))
    a = torch.arange(positions, dtype=torch.float64, device=device)[:, None] * f
    return a.cos().float(), a.sin().float()


class StackExecutor:
    def __init__(self, model):
        self.model = model
        self.cfg = model.config
        self.runs = self.cfg.runs()
        self.kv_src = self.cfg.kv_sources()
        self._mix = {RGLRUMixer: self._rglru, ParallelMixer: self._parallel, RotaryAttention: self._rotary,
                     TokenShiftMemory: self._shift_memory, ForgetGateMemory: self._forget_memory}
        self._rope: dict = {}       # kept for good: captured decode graphs point at the tables
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
            if isinstance(layer.mlp, PlainMLP):
                d["up"], _ = joint_weight([layer.mlp.up_proj])
            elif layer.mlp is not None:
                d["gu"], _ = joint_weight([layer.mlp.gate_proj, layer.mlp.up_proj])
            fresh.append(d)
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
            src = {k: d[k] for k in ("proj", "gates", "gu", "up") if k in d}
            if layer.mlp is not None:
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
        d, a, src = self.w[i], m.spec, self.kv_src[r]
        proj = linear(h, d["proj"], d["proj_bias"], packed=self.pk(i, "proj") if rb.decode else None)
        key = (a.rot_dims, a.rot_base, pool.max_pages * pool.page_size)
        if key not in self._rope:
            self._rope[key] = rope_table(key[2], a.rot_dims, a.rot_base, h.device)
        cos, sin = self._rope[key]
        nq, kv = a.heads * a.dim, 0 if a.kv_from is not None else a.kv_heads
        q = SK.rope_norm_write(proj, 0, nq, nq + kv * a.dim, cos, sin, a.rot_dims, m.eps, rb, pool.table, pool.page_size, a.heads,
                               kv, a.dim, a.vdim, pool.k[src], pool.v[src])
        att = self._attend(q, a, None, rb, pool, src)
        return (linear(att, m.o_proj.weight, m.o_proj.bias), None, None, None)

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

    def _few(self, x, w, rb: RaggedBatch, act: int, **rows) -> torch.Tensor:
        """act(x w^T) for narrow w."""
        if rb.decode and x.dtype == torch.bfloat16 and x.shape[1] % 8 == 0 and w.shape[0] <= FEW_OUTPUTS:
            return SK.few_outputs(x, w, act, **rows)
        return SK.small_act(linear(x, w, out_dtype=torch.float32), x.dtype, act, **rows)

    def _side(self, i, side, x, rb: RaggedBatch):
        dim = self.cfg.token_side
        y = self._few(x, side.gate_proj.weight, rb, SK.ACT_GELU_ROW, tokens=rb.tokens, rows=self.model.side_embed, col=i * dim)
        return (linear(y, side.proj.weight), None, side.norm.weight, None)

    def _attend(self, q, a, bias, rb: RaggedBatch, pool, r):
        """Tensor-core kernels where the heads fit them (the framework's paged decode and flash attention, extended by the
        bias and the kept tokens); otherwise, and in 32-bit, the general kernel."""
        fits = q.dtype == torch.bfloat16 and a.dim == a.vdim and a.dim in (64, 128, 256) and not self.plain
        kw = dict(scale=a.scale, softcap=a.softcap, window=a.window, chunk=a.chunk, keep_first=a.keep_first, bias=bias)
        if fits and rb.decode and a.heads // a.kv_heads <= 16:
            max_ctx = pool.table.shape[1] * pool.page_size
            span = min((s for s in (a.window, a.chunk) if s > 0), default=0)       # most keys a query sees besides the kept ones
            split = K.decode_split_tokens(rb.n, a.kv_heads, min(max_ctx, span + a.keep_first + 128) if span else max_ctx)
            return K.paged_decode(q.view(rb.n, a.heads, a.dim), pool.k[r], pool.v[r], pool.table, rb.slot, self._lens,
                                  num_kv_heads=a.kv_heads, page_size=pool.page_size, max_ctx=max_ctx, split_tokens=split,
                                  **kw).view(rb.n, -1)
        if fits and not rb.decode and pool.page_size % 64 == 0:
            return K.attn_fwd_paged(q, pool.k[r], pool.v[r], rb, pool.table, pool.page_size, num_heads=a.heads,
                                    num_kv_heads=a.kv_heads, head_dim=a.dim, **kw)
        return SK.window_attn(q, pool.k[r], pool.v[r], rb, pool.table, pool.page_size, a, bias)

    def _mlp(self, i, mlp, h, rb: RaggedBatch):
        if isinstance(mlp, PlainMLP):
            pup = self.pk(i, "up") if rb.decode else None
            act = K.gemm_packed(h, pup, xielu=mlp.act) if pup is not None else SK.xielu_(linear(h, self.w[i]["up"]), mlp.act)
            return linear(act, mlp.down_proj.weight, packed=self.pk(i, "down") if rb.decode else None)
        gu_w = self.w[i]["gu"]
        F = gu_w.shape[0] // 2
        pgu = self.pk(i, "gu") if rb.decode else None
        if pgu is not None and pgu.glu:
            act = K.gemm_packed(h, pgu, glu=K.GLU_SILU)
        else:
            gu = linear(h, gu_w, packed=pgu)
            act = K.glu_fwd(gu[:, :F], gu[:, F:], K.GLU_SILU) if gu.dtype == torch.bfloat16 and F % 8 == 0 else SK.silu_mul(gu)
        return linear(act, mlp.down_proj.weight, packed=self.pk(i, "down") if rb.decode else None)

    # ------------------------------------------------------------------------------------------------ the stack
    @torch.no_grad()
    def forward(self, rb: RaggedBatch, pool, layer_sums: Optional[list] = None) -> torch.Tensor:
        """Final normed hidden rows [n, D] of the batch's tokens. `pool`: the engine's PagePool (cache, page table, states).
        `layer_sums` (a list) receives the sum of the streams after every layer pass."""
        cfg, model = self.cfg, self.model
        eps, n = cfg.norm_eps, rb.n
        x = torch.empty((n, max(cfg.streams, 1), cfg.embed_dim), dtype=torch.float32, device=rb.tokens.device)
        close = dict(tokens=rb.tokens, embed=model.embed_tokens,       # what the next stream_step closes
                     embed_w=None if model.embed_norm is None else model.embed_norm.weight)

        def pending(out, hc):
            y, y2, wy, wy2 = out
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
            return SK.stream_step(x, eps, groups=cfg.norm_groups, w_in=w_in, norm_w=norm_w, sum_out=total, **close, **kw)

        for r, i in enumerate(self.runs):
            layer = model.layers[i]
            shifts = rb.decode and isinstance(layer.mixer, TokenShiftMemory)
            h = step(self._hc(layer.hc1)[0], layer.input_layernorm.weight,
                     **(dict(shift=(self.w[i]["mu"], pool.state[r]["last"]), rb=rb) if shifts else {}))
            close = pending(self._mix[type(layer.mixer)](i, layer.mixer, h, rb, pool, r), layer.hc1)
            if layer.mlp is not None:
                h = step(self._hc(layer.hc2)[0], layer.post_attention_layernorm.weight)
                close = pending((self._mlp(i, layer.mlp, h, rb), None, None, None), layer.hc2)
            if layer.side is not None:
                close = pending(self._side(i, layer.side, step(None, None, raw=True), rb), None)
            ended = True
        return step(None, model.norm.weight)

    def logits(self, hidden: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """fp32 logits of normed hidden rows."""
        packed = self.pk(len(self.model.layers), "head")
        if hidden.dtype == torch.bfloat16 and packed is not None:
            return K.gemm_packed(hidden, packed, out=out, out_dtype=torch.float32)
        if hidden.dtype == torch.bfloat16 and hidden.shape[1] % 8 == 0:
            return K.gemm(hidden, self.model.head_weight(), out=out, out_dtype=torch.float32)
        z = linear(hidden, self.model.head_weight(), out_dtype=torch.float32)
        return z if out is None else out.copy_(z)
