"""Launchers of the layer-stack kernels (csrc/stack.cu, recurrent.cu, window_attention.cu). Activations and weights are
bf16 or float (the `dtype` argument of the entry points), residual streams, states and gates fp32."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _lib
from .kernels import _count
from .ragged import RaggedBatch

_P, _I, _LL, _F = _lib.P, _lib.I, _lib.LL, _lib.F
_RB = [_P, _P, _P, _P, _I, _I]
_lib.register_cuda_sigs({
    "tb_stream_step": [_I, _P, _I, _I, _I, _F, _P, _P, _P, _P, _P, _P, _P, _P, _I, _P, _P, _P, _P, _P],
    "tb_few_outputs": [_P, _P, _I, _I, _I, _P, _P],
    "tb_silu_mul": [_I, _P, _P, _LL, _I, _P],
    "tb_gate_outputs": [_I, _P, _P, _P, _LL, _I, _I, _P, _F, _I, _I, _I, _I, _P, _P, _P],
    "tb_rglru": [_I, _P, _LL, _I, _I, _P, _P, _P, _P, _P, _P, _P, *_RB, _I, _I, _I, _P, _P, _P, _P, _P, _P, _I, _P, _P,
                 _P, _I, _P, _P, _P],
    "tb_mlstm_slices": [_I],
    "tb_mlstm": [_I, _P, _LL, _I, _I, _I, _P, _P, _P, _F, *_RB, _I, _I, _I, _P, _P, _P, _P, _I, _I, _P],
    "tb_qk_norm_write": [_I, _P, _LL, _I, _I, _I, _P, _P, _F, *_RB, _P, _I, _I, _I, _I, _I, _P, _P, _P, _P],
    "tb_window_attn": [_I, _P, _P, _P, *_RB, _P, _I, _I, _I, _I, _I, _I, _F, _P, _I, _I, _I, _P, _P],
})


def _dt(t: torch.Tensor) -> int:
    if t.dtype == torch.bfloat16:
        return 0
    if t.dtype == torch.float32:
        return 1
    raise TypeError(f"layer-stack kernels run bf16 or float32, not {t.dtype}")


def stream_step(x: torch.Tensor, eps: float, *, y=None, y2=None, wy=None, wy2=None, mix=None, w_out=None, tokens=None, embed=None,
                w_in=None, norm_w=None, sum_out: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """Close one sublayer (y [, y2 with their norms], mix, w_out; or start from the embedding rows of `tokens`) and open
    the next: returns h = norm(sum_s w_in[s] x_s) * norm_w (w_in None: the plain sum; norm_w None: nothing follows).
    x fp32 [n, S, D] is updated in place; `sum_out` fp32 [n, D] receives the sum of the streams."""
    n, S, D = x.shape
    ref = norm_w if norm_w is not None else (y if y is not None else embed)
    h = torch.empty((n, D), dtype=ref.dtype, device=x.device) if norm_w is not None else None
    rc = _lib.cuda().tb_stream_step(_dt(ref), x.data_ptr(), n, S, D, float(eps), _lib.ptr(y), _lib.ptr(y2), _lib.ptr(wy),
                                    _lib.ptr(wy2), _lib.ptr(mix), _lib.ptr(w_out), _lib.ptr(tokens), _lib.ptr(embed),
                                    0 if embed is None else embed.shape[0], _lib.ptr(w_in), _lib.ptr(norm_w), _lib.ptr(h),
                                    _lib.ptr(sum_out), _lib.stream_ptr())
    _lib.check(rc, "tb_stream_step")
    _count()
    return h


def silu_mul(gu: torch.Tensor) -> torch.Tensor:
    """gu [rows, 2 F] -> silu(gu[:, :F]) * gu[:, F:], any F."""
    rows, F2 = gu.shape
    h = torch.empty((rows, F2 // 2), dtype=gu.dtype, device=gu.device)
    rc = _lib.cuda().tb_silu_mul(_dt(gu), gu.data_ptr(), h.data_ptr(), rows, F2 // 2, _lib.stream_ptr())
    _lib.check(rc, "tb_silu_mul")
    _count()
    return h


def few_outputs(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x bf16 [n, K] @ w^T [N, K] -> fp32 [n, N] for a handful of outputs and decode-size n (a GEMM tile would leave one CTA
    with the whole contraction)."""
    assert x.dtype == w.dtype == torch.bfloat16 and x.is_contiguous() and w.is_contiguous() and x.shape[1] % 8 == 0
    out = torch.empty((x.shape[0], w.shape[0]), dtype=torch.float32, device=x.device)
    rc = _lib.cuda().tb_few_outputs(x.data_ptr(), w.data_ptr(), x.shape[0], x.shape[1], w.shape[0], out.data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "tb_few_outputs")
    _count()
    return out


def gate_outputs(attn, o, proj, g1_off: int, g2_off: int, norm_w, eps: float, heads: int, vdim: int):
    """attn [n, C1] * sigmoid(g1), and o fp32 [n, heads, vdim] normed per head * norm_w * sigmoid(g2)."""
    n, C1 = attn.shape
    a1 = torch.empty_like(attn)
    a2 = torch.empty((n, heads * vdim), dtype=attn.dtype, device=attn.device)
    rc = _lib.cuda().tb_gate_outputs(_dt(attn), attn.data_ptr(), o.data_ptr(), proj.data_ptr(), proj.stride(0), g1_off, g2_off,
                                     norm_w.data_ptr(), float(eps), n, C1, heads, vdim, a1.data_ptr(), a2.data_ptr(),
                                     _lib.stream_ptr())
    _lib.check(rc, "tb_gate_outputs")
    _count()
    return a1, a2


def rglru(proj, x_off: int, y_off: int, m, rb: RaggedBatch, state: dict, plain: bool = False) -> torch.Tensor:
    """Convolution, gates, recurrence and output gate of `models.mixers.RGLRUMixer` m on its projections; [n, W].
    `plain`: the simple kernels of the 32-bit path, also for bf16."""
    n, sp = proj.shape[0], m.spec
    W = sp.width
    dev = proj.device
    one = rb.decode and not plain and proj.dtype == torch.bfloat16
    tiles = (None, None, None, 0) if plain or one or proj.dtype != torch.bfloat16 else rb.tiles()
    out = torch.empty((n, W), dtype=proj.dtype, device=dev)
    u = torch.empty_like(out)
    ws = torch.empty((2 * n + 2 * tiles[3], W), dtype=torch.float32, device=dev)
    A, Bv, LH, LP = ws[:n], ws[n:2 * n], ws[2 * n:2 * n + tiles[3]], ws[2 * n + tiles[3]:]
    rc = _lib.cuda().tb_rglru(_dt(proj), proj.data_ptr(), proj.stride(0), x_off, y_off, m.conv_weight.data_ptr(),
                              m.conv_bias.data_ptr(), m.ra_weight.data_ptr(), m.ra_bias.data_ptr(), m.ri_weight.data_ptr(),
                              m.ri_bias.data_ptr(), m.lam.data_ptr(), *rb.args(), W, sp.conv, sp.blocks, state["s"].data_ptr(),
                              state["ring"].data_ptr(), u.data_ptr(), A.data_ptr(), Bv.data_ptr(), out.data_ptr(), int(one),
                              _lib.ptr(tiles[0]), _lib.ptr(tiles[1]), _lib.ptr(tiles[2]), tiles[3], LH.data_ptr(), LP.data_ptr(),
                              _lib.stream_ptr())
    _lib.check(rc, "tb_rglru")
    _count(1 if one else 4)
    return out


def mlstm(proj, q_off: int, k_off: int, v_off: int, gates, i_bias, f_bias, cap: float, rb: RaggedBatch, heads: int, dk: int,
          dv: int, state: dict, plain: bool = False) -> torch.Tensor:
    """Matrix memory over a ragged batch; gates fp32 [n, 2 heads] (may be overwritten). Returns o fp32
    [n, heads, dv]. `plain`: the token by
    token kernel of the 32-bit path, also for bf16."""
    n = proj.shape[0]
    assert gates.dtype == torch.float32 and gates.is_contiguous() and gates.shape == (n, 2 * heads)
    out = torch.empty((n, heads, dv), dtype=torch.float32, device=proj.device)
    rc = _lib.cuda().tb_mlstm(_dt(proj), proj.data_ptr(), proj.stride(0), q_off, k_off, v_off, gates.data_ptr(),
                              i_bias.data_ptr(), f_bias.data_ptr(), float(cap), *rb.args(), heads, dk, dv,
                              state["S"].data_ptr(), state["n"].data_ptr(), state["m"].data_ptr(), out.data_ptr(),
                              int(rb.decode and not plain), int(not plain), _lib.stream_ptr())
    _lib.check(rc, "tb_mlstm")
    _count()
    return out


def qk_norm_write(proj, q_off: int, k_off: int, v_off: int, q_w, k_w, eps: float, rb: RaggedBatch, table, page_size: int,
                  k_pool, v_pool, NQ: int) -> torch.Tensor:
    """Whole-projection RMS norm of q and k; q [n, NQ] is returned, k and v rows go to their pages."""
    n = proj.shape[0]
    q = torch.empty((n, NQ), dtype=proj.dtype, device=proj.device)
    rc = _lib.cuda().tb_qk_norm_write(_dt(proj), proj.data_ptr(), proj.stride(0), q_off, k_off, v_off, q_w.data_ptr(),
                                      k_w.data_ptr(), float(eps), *rb.args(), table.data_ptr(), table.shape[1], page_size, NQ,
                                      k_pool.shape[-1], v_pool.shape[-1], q.data_ptr(), k_pool.data_ptr(), v_pool.data_ptr(),
                                      _lib.stream_ptr())
    _lib.check(rc, "tb_qk_norm_write")
    _count()
    return q


def window_attn(q, k_pool, v_pool, rb: RaggedBatch, table, page_size: int, sp, bias) -> torch.Tensor:
    """`sp`: models.mixers.WindowAttentionSpec; bias fp32 [heads, far + 1]. Returns [n, heads * vdim]."""
    n = q.shape[0]
    out = torch.empty((n, sp.heads * sp.vdim), dtype=q.dtype, device=q.device)
    rc = _lib.cuda().tb_window_attn(_dt(q), q.data_ptr(), k_pool.data_ptr(), v_pool.data_ptr(), *rb.args(), table.data_ptr(),
                                    table.shape[1], page_size, sp.heads, sp.kv_heads, sp.dim, sp.vdim, float(sp.scale),
                                    bias.data_ptr(), bias.shape[1] - 1, sp.window, sp.keep_first, out.data_ptr(),
                                    _lib.stream_ptr())
    _lib.check(rc, "tb_window_attn")
    _count()
    return out
