"""Launchers of the layer-stack kernels (csrc/stack.cu, recurrent.cu, linear_attention.cu, window_attention.cu,
latent_attention.cu, moe_infer.cu). Activations and weights are bf16 or float (the `dtype` argument of the entry points), residual streams, states and gates fp32."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _lib
from . import kernels as K
from .kernels import _count
from .ragged import RaggedBatch

_P, _I, _LL, _F = _lib.P, _lib.I, _lib.LL, _lib.F
_RB = [_P, _P, _P, _P, _I, _I]
_lib.register_cuda_sigs({
    "tb_stream_step": [_I, _P, _I, _I, _I, _F, _P, _P, _P, _P, _P, _P, _P, _P, _I, _P, _F, _P, _I, _I, _P, _P, _P, _LL, _P, _P, _I, _P, _P,
                       _P, _LL, _LL, _LL, _P, _P, _LL, _P, _P, _P, _P, _P, _P, _P],
    "tb_few_outputs": [_P, _P, _I, _I, _I, _I, _P, _I, _P, _LL, _I, _P, _I, _P],
    "tb_small_act": [_I, _P, _I, _I, _I, _P, _I, _P, _LL, _I, _P, _P],
    "tb_token_shift": [_I, _P, _P, _I, _P, *_RB, _I, _P, _P],
    "tb_xielu": [_I, _P, _P, _LL, _P],
    "tb_gated_linear": [_I, _I, _P, _LL, _P, _LL, _P, _LL, _P, _LL, _P, _LL, _P, _LL, _P, _I, _P, _P, _F, _F, *_RB, _I, _I, _I, _P, _P,
                        _P, _I, _P, _I, _F, _F, _P, _P, _LL, _I, _I, _P],
    "tb_glu": [_I, _I, _P, _P, _LL, _LL, _I, _P],
    "tb_keep_last": [_I, _P, _P, *_RB, _I, _P],
    "tb_gate_outputs": [_I, _P, _P, _P, _LL, _I, _I, _P, _F, _I, _I, _I, _I, _P, _P, _P],
    "tb_rglru": [_I, _P, _LL, _I, _I, _P, _P, _P, _P, _P, _P, _P, *_RB, _I, _I, _I, _P, _P, _P, _P, _P, _P, _I, _P, _P,
                 _P, _I, _P, _P, _P],
    "tb_mlstm_slices": [_I],
    "tb_mlstm": [_I, _P, _LL, _I, _I, _I, _P, _P, _P, _F, *_RB, _I, _I, _I, _P, _P, _P, _P, _I, _I, _P],
    "tb_qk_norm_write": [_I, _P, _LL, _I, _I, _I, _P, _P, _F, *_RB, _P, _I, _I, _I, _I, _I, _P, _P, _P, _P],
    "tb_rope_norm_write": [_I, _P, _LL, _I, _I, _I, _P, _P, _P, _P, _I, _I, _F, _I, *_RB, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P, _P, _P, _P],
    "tb_window_attn": [_I, _P, _LL, _I, _P, _P, *_RB, _P, _I, _I, _I, _I, _I, _I, _I, _I, _F, _F, _P, _I, _I, _I, _I, _F, _P, _P, _LL,
                       _F, _P, _LL, _P],
    "tb_latent_write": [_I, _P, _LL, _I, _I, _I, _I, _I, _P, _F, _P, _P, _I, *_RB, _P, _I, _I, _I, _P, _P],
    "tb_latent_gather": [_P, _P, _P, _I, _P, _I, _I, _I, _P, _P],
    "tb_head_product": [_I, _P, _LL, _I, _P, _P, _I, _I, _I, _P, _LL, _I, _P, _I, _I, _I, _P],
    "tb_latent_decode": [_P, _P, _LL, _P, _I, _I, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P, _I, _P, _P, _P, _P, _P],
    "tb_moe_route": [_I, _P, _P, *_RB, _I, _I, _P, _P, _P, _P, _P, _P],
    "tb_moe_route_lists": [_I, _P, _P, *_RB, _I, _I, _P, _P, _P, _P, _P],
    "tb_moe_experts": [_I, _I, _P, _LL, _P, _P, _I, _I, _I, _I, _I, _P, _P, _P, _P, _P, _P, _P, _P],
})


def _dt(t: torch.Tensor) -> int:
    if t.dtype == torch.bfloat16:
        return 0
    if t.dtype == torch.float32:
        return 1
    raise TypeError(f"layer-stack kernels run bf16 or float32, not {t.dtype}")


def stream_step(x: torch.Tensor, eps: float, *, y=None, y2=None, wy=None, wy2=None, mix=None, w_out=None, tokens=None, embed=None,
                embed_w=None, embed_scale: float = 1.0, pos=None, pairs=None, start_out=None, groups: int = 1, w_in=None, norm_w=None,
                raw: bool = False, out=None, shift=None, both: bool = False, keep=None, rb: Optional[RaggedBatch] = None,
                sum_out: Optional[torch.Tensor] = None):
    """Close one sublayer (y [, y2 with their norms; y alone with its norm wy], mix, w_out; or start from the embedding rows
    of `tokens`, normed with embed_w if given, times embed_scale, plus the rows `pos` [positions, D] of the tokens' positions in
    the batch `rb`; or both: the embedding rows are added to every stream after the sublayer, not to sum_out) and open the next: returns h = norm(sum_s w_in[s] x_s) * norm_w (w_in None:
    the plain sum; norm_w None: nothing follows, or with `raw` the sum itself). The norms of rows and embeddings are taken
    over `groups` equal parts. x fp32 [n, S, D] is updated in place; `sum_out` fp32 [n, D] receives the sum of the streams.
    `shift` = (mu [m, D], carry fp32 [slots, D]), for batches `rb` of single tokens: returns the m mixes
    h + (carry - h) mu [m, n, D] instead of h (`both`: beside it) and replaces the slots' carry by h.
    `pairs` = (table [buckets + 1, D], (buckets, p, c), last int64 [slots]): the embedding also has the table's row
    (p * token before + c * token) mod buckets, `last` holding the tokens before the entries' first ones; a sequence's first token
    takes the last row. `start_out`: columns that take the embedding rows as they are added. `out`: columns of wider rows for h.
    `keep` int64 [slots] receives every entry's last token."""
    n, S, D = x.shape
    ref = norm_w if norm_w is not None else (y if y is not None else embed)
    mu, carry = shift or (None, None)
    mixes = torch.empty((mu.shape[0], n, D), dtype=ref.dtype, device=x.device) if shift else None
    h = out
    if h is None and ((norm_w is not None and (not shift or both)) or raw):
        h = torch.empty((n, D), dtype=ref.dtype, device=x.device)
    table, (buckets, m_prev, m_cur), last = pairs or (None, (0, 0, 0), None)
    rc = _lib.cuda().tb_stream_step(_dt(ref), x.data_ptr(), n, S, D, float(eps), _lib.ptr(y), _lib.ptr(y2), _lib.ptr(wy),
                                    _lib.ptr(wy2), _lib.ptr(mix), _lib.ptr(w_out), _lib.ptr(tokens), _lib.ptr(embed),
                                    0 if embed is None else embed.shape[0], _lib.ptr(embed_w), float(embed_scale), _lib.ptr(pos),
                                    0 if pos is None else pos.shape[0], int(groups), _lib.ptr(w_in), _lib.ptr(norm_w), _lib.ptr(h),
                                    0 if h is None else h.stride(0), _lib.ptr(sum_out), _lib.ptr(mu), 0 if mu is None else mu.shape[0],
                                    _lib.ptr(carry), _lib.ptr(mixes), _lib.ptr(table), buckets, m_prev, m_cur, _lib.ptr(last),
                                    _lib.ptr(start_out), 0 if start_out is None else start_out.stride(0), _lib.ptr(keep),
                                    0 if keep is None else rb.tokens.data_ptr(),
                                    *((0, 0, 0, 0) if rb is None else rb.args()[:4]), _lib.stream_ptr())
    _lib.check(rc, "tb_stream_step")
    _count()
    return (h, mixes) if both else mixes if shift else h


def token_shift(h, mu, carry, rb: RaggedBatch) -> torch.Tensor:
    """h [n, D] + (row of the token before - h) * mu[m] -> [m, n, D]; the row before a portion is its slot's `carry` (zero at
    the start of a sequence). The carry is replaced by the recurrence that runs on the mixes."""
    n, D = h.shape
    assert h.is_contiguous() and mu.is_contiguous()
    mixes = torch.empty((mu.shape[0], n, D), dtype=h.dtype, device=h.device)
    rc = _lib.cuda().tb_token_shift(_dt(h), h.data_ptr(), mu.data_ptr(), mu.shape[0], carry.data_ptr(), *rb.args(), D,
                                    mixes.data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "tb_token_shift")
    _count()
    return mixes


def keep_last(h, carry, rb: RaggedBatch) -> None:
    """carry fp32 [slots, D] of the batch's slots = the last rows of its entries in h [n, D]."""
    assert h.is_contiguous()
    rc = _lib.cuda().tb_keep_last(_dt(h), h.data_ptr(), carry.data_ptr(), *rb.args(), h.shape[1], _lib.stream_ptr())
    _lib.check(rc, "tb_keep_last")
    _count()


def xielu_(x: torch.Tensor, act: torch.Tensor) -> torch.Tensor:
    """xIELU in place, act = its two numbers (before softplus)."""
    assert x.is_contiguous() and act.dtype == x.dtype
    rc = _lib.cuda().tb_xielu(_dt(x), x.data_ptr(), act.data_ptr(), x.numel(), _lib.stream_ptr())
    _lib.check(rc, "tb_xielu")
    _count()
    return x


def glu(gu: torch.Tensor, kind: int, out=None) -> torch.Tensor:
    """gu [rows, 2 F] -> act(gu[:, :F]) * gu[:, F:], any F; kind: K.GLU_SILU or K.GLU_GELU. `out`: columns of wider rows."""
    rows, F2 = gu.shape
    assert gu.is_contiguous()
    h = torch.empty((rows, F2 // 2), dtype=gu.dtype, device=gu.device) if out is None else out
    rc = _lib.cuda().tb_glu(_dt(gu), kind, gu.data_ptr(), h.data_ptr(), h.stride(0), rows, F2 // 2, _lib.stream_ptr())
    _lib.check(rc, "tb_glu")
    _count()
    return h


ACT_NONE, ACT_TANH, ACT_GELU_ROW = 0, 1, 2      # csrc/stack.cu: apply_small


def few_outputs(x: torch.Tensor, w: torch.Tensor, act: int = ACT_NONE, tokens=None, rows=None, col: int = 0) -> torch.Tensor:
    """act(x bf16 [n, K] @ w^T [N, K]) for few outputs and decode-size n (GEMM tiles would leave a few CTAs with the whole
    contraction): fp32 [n, N], or bf16 after an activation. ACT_GELU_ROW multiplies by columns col .. col + N of the
    tokens' rows of the table `rows`."""
    assert x.dtype == w.dtype == torch.bfloat16 and x.is_contiguous() and w.is_contiguous() and x.shape[1] % 8 == 0
    out = torch.empty((x.shape[0], w.shape[0]), dtype=torch.float32 if act == ACT_NONE else torch.bfloat16, device=x.device)
    rc = _lib.cuda().tb_few_outputs(x.data_ptr(), w.data_ptr(), x.shape[0], x.shape[1], w.shape[0], act, _lib.ptr(tokens),
                                    0 if rows is None else rows.shape[0], _lib.ptr(rows), 0 if rows is None else rows.shape[1],
                                    col, out.data_ptr(), int(act != ACT_NONE), _lib.stream_ptr())
    _lib.check(rc, "tb_few_outputs")
    _count()
    return out


def small_act(z: torch.Tensor, dtype, act: int, tokens=None, rows=None, col: int = 0) -> torch.Tensor:
    """The activations of `few_outputs` on fp32 products z [n, N] of any size."""
    assert z.dtype == torch.float32 and z.is_contiguous()
    out = torch.empty(z.shape, dtype=dtype, device=z.device)
    rc = _lib.cuda().tb_small_act(_dt(out), z.data_ptr(), z.shape[0], z.shape[1], act, _lib.ptr(tokens),
                                  0 if rows is None else rows.shape[0], _lib.ptr(rows), 0 if rows is None else rows.shape[1], col,
                                  out.data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "tb_small_act")
    _count()
    return out


GATES_BONUS, GATES_LOWER, GATES_ROOT = 0, 1, 2  # csrc/linear_attention.cu: Mode
STEP_WIDTH = 256        # heads with wider values may not fit the decode kernel and take the token by token one


def gated_linear(mode: int, q, k, v, z, c0, c1, rb: RaggedBatch, heads: int, dk: int, dv: int, state, norm_w, eps: float, *,
                 gate=None, per_head: bool = False, carry=None, h=None, plain: bool = False, low_rank=None, q_scale: float = 1.0,
                 tau: float = 1.0, out=None, out_scale: float = 1.0) -> torch.Tensor:
    """Matrix state with a decay per head and channel over a ragged batch, its head norm and output gate; [n, heads * dv].
    GATES_BONUS: decay exp(-exp(z + c0)), keys k, bonus c1 for the current token. GATES_LOWER: decay
    c1 + (1 - c1) sigmoid(z + c0), key 1 - decay, silu(q). GATES_ROOT: decay sigmoid(z + c0)^(1 / tau), keys k, q * q_scale.
    q, k, v, gate: column views of rows [n, ..]; z fp32, or None with `low_rank` = (x [n, rank], w [heads * dk, rank]) in a decode
    step: z = x w^T, formed in the kernel. norm_w [dv], or [heads * dv] with per_head. carry / h: see `token_shift` (portions
    only). `out`: columns of wider rows; the result is scaled by out_scale.
    `plain`: the token by token kernel of the 32-bit path, also for bf16."""
    n = q.shape[0]
    x, w2 = low_rank if z is None else (None, None)
    assert (z is None or z.dtype == torch.float32) and all(t is None or t.stride(1) == 1 for t in (q, k, v, z, x, gate, out))
    one = rb.decode and not plain
    raw = torch.empty((n, heads * dv), dtype=torch.float32, device=q.device) if not one or dv > STEP_WIDTH else None
    if out is None:
        out = torch.empty((n, heads * dv), dtype=q.dtype, device=q.device)
    ld = lambda t: 0 if t is None else t.stride(0)  # noqa: E731
    if rb.decode:
        carry = h = None                        # the launch that made the mixes has replaced it
    rc = _lib.cuda().tb_gated_linear(_dt(q), mode, q.data_ptr(), ld(q), _lib.ptr(k), ld(k), v.data_ptr(), ld(v), _lib.ptr(gate),
                                     ld(gate), _lib.ptr(z), ld(z), _lib.ptr(x), ld(x), _lib.ptr(w2), 0 if x is None else x.shape[1],
                                     c0.data_ptr(), _lib.ptr(c1), float(q_scale), 1.0 / tau, *rb.args(), heads, dk, dv,
                                     state.data_ptr(), _lib.ptr(h), _lib.ptr(carry), 0 if h is None else h.shape[1],
                                     norm_w.data_ptr(), int(per_head), float(eps), float(out_scale), _lib.ptr(raw), out.data_ptr(),
                                     out.stride(0), int(one), int(not plain), _lib.stream_ptr())
    _lib.check(rc, "tb_gated_linear")
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


def rope_norm_write(proj, q_off: int, k_off: int, v_off: int, cos, sin, rot_dims: int, eps: float, rb: RaggedBatch, table,
                    page_size: int, heads: int, kv_heads: int, dim: int, vdim: int, k_pool, v_pool, *, q_w=None, k_w=None,
                    interleaved: bool = False, stored: Optional[tuple] = None, norm_qk: bool = True, norm_v: bool = False) -> torch.Tensor:
    """Every query and key head divided by its root mean square (times q_w / k_w [dim]) and its first rot_dims dimensions turned
    (cos / sin fp32 [positions, rot_dims / 2]; halves of them together, or neighbours if `interleaved`); q is returned, k and v
    rows go to their pages. `stored`: widths the key / value heads are kept at, with zeros behind them (queries like keys; default:
    as they are). kv_heads 0: the rows hold queries only and nothing is written; heads 0: keys and values only. `norm_qk`, `norm_v`:
    whether query and key heads / value heads are divided by their root mean square."""
    n = proj.shape[0]
    wq, wv = stored or (dim, vdim)
    q = torch.empty((n, heads * wq), dtype=proj.dtype, device=proj.device)
    rc = _lib.cuda().tb_rope_norm_write(_dt(proj), proj.data_ptr(), proj.stride(0), q_off, k_off, v_off, _lib.ptr(q_w), _lib.ptr(k_w),
                                        _lib.ptr(cos), _lib.ptr(sin), rot_dims, int(interleaved), float(eps),
                                        int(norm_qk) + 2 * int(norm_v), *rb.args(),
                                        table.data_ptr(), table.shape[1], page_size, heads, kv_heads, dim, vdim, wq, wv, q.data_ptr(),
                                        k_pool.data_ptr(), v_pool.data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "tb_rope_norm_write")
    _count()
    return q


def window_attn(q, k_pool, v_pool, rb: RaggedBatch, table, page_size: int, sp, bias, out=None, out_scale: float = 1.0, sinks=None,
                gate=None, sizes: Optional[tuple] = None) -> torch.Tensor:
    """`sp`: an attention spec of models.mixers; bias fp32 [heads, far + 1] or None; `sinks` fp32 [heads], `gate` [n, heads] as in
    kernels.paged_decode. q [n, heads * stored], or a view [n, heads, ..]. Returns out_scale * [n, heads * vdim]; `out`: columns of wider
    rows. `sizes`: other (key heads, key size, value size, stored key, stored value) than the spec's."""
    n = q.shape[0]
    G, dq, dv, wq, wv = sizes or (sp.kv_heads, sp.dim, sp.vdim, *sp.stored(q.dtype))
    if q.dim() == 2:
        q = q.view(n, sp.heads, wq)
    assert q.stride(2) == 1
    if out is None:
        out = torch.empty((n, sp.heads * dv), dtype=q.dtype, device=q.device)
    rc = _lib.cuda().tb_window_attn(_dt(q), q.data_ptr(), q.stride(0), q.stride(1), k_pool.data_ptr(), v_pool.data_ptr(), *rb.args(),
                                    table.data_ptr(), table.shape[1], page_size, sp.heads, G, dq, dv, wq, wv, float(sp.scale),
                                    float(sp.softcap), _lib.ptr(bias), 0 if bias is None else bias.shape[1] - 1, sp.window,
                                    sp.chunk, sp.keep_first, float(sp.sink), _lib.ptr(sinks), _lib.ptr(gate),
                                    0 if gate is None else gate.stride(0), float(out_scale), out.data_ptr(), out.stride(0),
                                    _lib.stream_ptr())
    _lib.check(rc, "tb_window_attn")
    _count()
    return out


# ------------------------------------------------------------------------------------------------ latents
def latent_write(proj, c_off: int, norm_w, cos, sin, rot_dims: int, eps: float, rb: RaggedBatch, table, page_size: int, heads: int, dim: int,
                 rot_dim: int, rank: int, pool) -> None:
    """proj [n, ..]: query heads of dim + rot_dim columns, and at c_off the latent (rank) and the shared key part (rot_dim). The
    first rot_dims of every rotated part turn (queries in place, halves together); the normed latent and the key part go to their
    page rows."""
    rc = _lib.cuda().tb_latent_write(_dt(proj), proj.data_ptr(), proj.stride(0), heads, dim, rot_dim, c_off, rank, norm_w.data_ptr(),
                                     float(eps), cos.data_ptr(), sin.data_ptr(), rot_dims, *rb.args(), table.data_ptr(), table.shape[1],
                                     page_size, pool.shape[-1], pool.data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "tb_latent_write")
    _count()


def latent_gather(pool, slot, pos, table, page_size: int) -> torch.Tensor:
    """[blocks * 64, W]: the cached rows of positions pos[i] .. pos[i] + 63 of the sequences in slot[i]."""
    out = torch.empty((slot.shape[0] * 64, pool.shape[-1]), dtype=pool.dtype, device=pool.device)
    rc = _lib.cuda().tb_latent_gather(pool.data_ptr(), slot.data_ptr(), pos.data_ptr(), slot.shape[0], table.data_ptr(), table.shape[1],
                                      page_size, pool.shape[-1], out.data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "tb_latent_gather")
    _count()
    return out


def head_product(x, w, out, *, transposed: bool = False, x_rows=None, out_rows=None, rows: int = 0, tail: int = 0) -> torch.Tensor:
    """out[t, h, :N] = x[t, h, :K] w[h], w bf16 [H, K, N] (or [H, N, K] `transposed`). x, out: views [.., H, ..] with free row and head
    strides; `x_rows` / `out_rows` int32 [rows] name their rows. `tail`: that many columns behind x's K are copied behind out's N,
    and what is left of out's columns becomes zero."""
    H = w.shape[0]
    K_, N = (w.shape[2], w.shape[1]) if transposed else (w.shape[1], w.shape[2])
    T = rows or x.shape[0]
    assert w.is_contiguous() and x.stride(2) == out.stride(2) == 1 and x.shape[2] >= K_ + tail and out.shape[2] >= N + tail
    rc = _lib.cuda().tb_head_product(int(not transposed), x.data_ptr(), x.stride(0), x.stride(1), _lib.ptr(x_rows), w.data_ptr(), H, K_, N,
                                     out.data_ptr(), out.stride(0), out.stride(1), _lib.ptr(out_rows), T, tail,
                                     0 if transposed else out.shape[2] - N, _lib.stream_ptr())
    _lib.check(rc, "tb_head_product")
    _count()
    return out


def latent_splits(tokens: int, heads: int, tiles: int) -> int:
    """Tiles of 64 keys per CTA of `latent_decode`: whole waves of one CTA per SM, each with a fixed cost of about two tiles, and about
    three for merging splits."""
    groups = -(-heads // (32 if heads > 16 else 16))
    cost = lambda per: -(-tokens * groups * -(-tiles // per) // 148) * (per + 2) + (3 if per < tiles else 0)  # noqa: E731
    return min(range(1, tiles + 1), key=lambda per: (cost(per), -per))


def latent_decode(q, pool, table, page_size: int, slots, lens, *, rank: int, scale: float, window: int, sinks, max_ctx: int,
                  split_tokens: int = 0) -> torch.Tensor:
    """Attention of single queries q bf16 [T, H, W] in the absorbed form over cached rows [pages, page_size, W], whose first `rank`
    columns are the values: bf16 [T, H, rank]. Query t sees the last `window` (0: all) of the first lens[t] rows of the
    sequence in slots[t]; sinks fp32 [H]."""
    T, H, W = q.shape
    assert q.is_contiguous() and pool.is_contiguous() and pool.shape[-1] == W
    tiles = -(-max_ctx // 64)
    if window > 0:
        tiles = min(tiles, -(-window // 64) + 1)
    per = split_tokens // 64 if split_tokens else latent_splits(T, H, tiles)
    splits = -(-tiles // per)
    ws = torch.empty(T * H * splits * (rank + 2) if splits > 1 else 0, dtype=torch.float32, device=q.device)
    out = torch.empty((T, H, rank), dtype=q.dtype, device=q.device)
    acc = T * H * splits * rank * 4
    rc = _lib.cuda().tb_latent_decode(q.data_ptr(), pool.data_ptr(), pool.shape[0] * page_size, table.data_ptr(), table.shape[1], page_size,
                                      slots.data_ptr(), lens.data_ptr(), T, H, rank, W, tiles, float(scale), int(window), _lib.ptr(sinks),
                                      per * 64, ws.data_ptr(), ws.data_ptr() + acc if splits > 1 else 0, out.data_ptr(),
                                      _lib.status_buffer(q.device).data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "tb_latent_decode")
    _count(1 if splits == 1 else 2)
    return out


# ------------------------------------------------------------------------------------------------ experts
ROWS_TOKENS = 128       # up to this many tokens an expert's weights are streamed past its few rows


def moe(h, logits, correction, gate_up, down, top: int, rb: RaggedBatch) -> torch.Tensor:
    """sum_j s_j expert_j(h) over the `top` experts with the largest score (+ correction [E] for the choice only); s: softmax of
    the fp32 router logits over all experts, not renormalised. gate_up [E, 2 F, D] (gate rows, then up rows), down [E, D, F];
    expert: down(silu(gate h) * up h). Returns [n, D] in h's type."""
    n, D = h.shape
    E, F2, _ = gate_up.shape
    F, dev = F2 // 2, h.device
    assert logits.dtype == torch.float32 and logits.shape == (n, E) and logits.is_contiguous() and h.stride(1) == 1
    assert gate_up.is_contiguous() and down.is_contiguous() and down.shape == (E, D, F)
    idx = torch.empty((n, top), dtype=torch.int32, device=dev)
    wts = torch.empty((n, top), dtype=torch.float32, device=dev)
    fits = h.dtype == torch.bfloat16 and D % 8 == 0 and F % 8 == 0 and h.stride(0) % 8 == 0 and h.data_ptr() % 16 == 0
    if fits and n > ROWS_TOKENS:
        hist = torch.empty((-(-n // 128), E), dtype=torch.int32, device=dev)
        seg = torch.empty(E + 1, dtype=torch.int32, device=dev)
        pos = torch.empty((n, top), dtype=torch.int32, device=dev)
        rc = _lib.cuda().tb_moe_route(_dt(h), logits.data_ptr(), _lib.ptr(correction), *rb.args(), E, top, idx.data_ptr(), wts.data_ptr(),
                                      hist.data_ptr(), seg.data_ptr(), pos.data_ptr(), _lib.stream_ptr())
        _lib.check(rc, "tb_moe_route")
        _count(3)
        rows = (n * top + E * 127 + 127) // 128 * 128
        xp = torch.empty((rows, D), dtype=h.dtype, device=dev)
        K.moe_scatter_rows(h, pos, None, xp)
        gu = torch.empty((rows, F2), dtype=h.dtype, device=dev)
        K.gemm_grouped(xp, gate_up.view(E * F2, D), gu, F2, K.moe_tiles_rows(seg, rows, F2, D, F2))
        y = K.gemm_grouped(K.glu_fwd(gu[:, :F], gu[:, F:], K.GLU_SILU), down.view(E * D, F), xp, D, K.moe_tiles_rows(seg, rows, D, F, D))
        return K.moe_gather_sum(y, pos, wts)
    off = torch.empty(E + 1, dtype=torch.int32, device=dev)
    order = torch.empty(n * top, dtype=torch.int32, device=dev)
    rc = _lib.cuda().tb_moe_route_lists(_dt(h), logits.data_ptr(), _lib.ptr(correction), *rb.args(), E, top, idx.data_ptr(),
                                        wts.data_ptr(), off.data_ptr(), order.data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "tb_moe_route_lists")
    act = torch.empty((n * top, F), dtype=h.dtype, device=dev)
    y = torch.empty((n * top, D), dtype=torch.float32, device=dev)
    out = torch.empty((n, D), dtype=h.dtype, device=dev)
    rc = _lib.cuda().tb_moe_experts(_dt(h), int(fits), h.data_ptr(), h.stride(0), gate_up.data_ptr(), down.data_ptr(), n, D, F, E, top,
                                    idx.data_ptr(), wts.data_ptr(), off.data_ptr(), order.data_ptr(), act.data_ptr(), y.data_ptr(),
                                    out.data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "tb_moe_experts")
    _count(4)
    return out
