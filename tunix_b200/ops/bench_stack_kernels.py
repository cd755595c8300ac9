"""Micro-benchmarks of the layer-stack kernels: `python -m tunix_b200.ops.bench_kernels stack [--model roluzen_8b|tovalix_8b|zikezen_8b|zigipel_8b]
[--batch 4 --seq 4096] [--decode-batch 64 --decode-ctx 1024] [--only mlstm_prefill,...]`.

One JSON line per kernel at the sizes of a preset: median time with L2 flushed between iterations, the algorithmic bytes and
operations (every input read once, every output written once; no repeated or split work counted), and the fraction of the
roofline, i.e. the larger of bytes / copy bandwidth and operations / GEMM throughput over the measured time. The like kernels
of uniform decoders (flash attention with the same window as a prefill calls it, paged decode, RMS norm, gated activation,
expert layer) come beside them."""
from __future__ import annotations

import json

import torch


def reporter(args, peaks, timer):
    peak_tf, peak_gb, which = peaks
    only = set(args.only.split(",")) if args.only else None

    def report(name, fn, nbytes, flops=0.0, note=None):
        if only and name not in only:
            return
        ms = timer(fn, args.iters, args.warmup)
        roof = max(nbytes / peak_gb / 1e6, flops / peak_tf / 1e9)
        line = {"kernel": name, "model": args.model, "ms": ms, "gbs": nbytes / ms / 1e6, "tflops": flops / ms / 1e9,
                "roofline_ms": roof, "frac_of_roofline": roof / ms, "peaks": which}
        if note:
            line["note"] = note
        print(json.dumps(line), flush=True)
    return report


def phases(args):
    """(phase, batch, entries, context) of a prefill and a decode step."""
    from .ragged import RaggedBatch
    for phase, ls in (("prefill", [args.seq] * args.batch), ("decode", [1] * args.decode_batch)):
        ctx = args.decode_ctx if phase == "decode" else args.seq
        work = [(i, ctx - 1 if phase == "decode" else 0, [1] * L) for i, L in enumerate(ls)]
        yield phase, RaggedBatch.build(work, torch.device("cuda")), len(ls), ctx


def page_pool(B, ctx, k_cols, v_cols):
    pages = -(-ctx // 64)
    mk = lambda n: torch.randn(B * pages, 64, n, device="cuda").to(torch.bfloat16)  # noqa: E731
    return mk(k_cols), mk(v_cols), torch.randperm(B * pages, device="cuda").int().view(B, pages)


def run(args, peaks, timer) -> None:
    from ..models.config import get_config
    family = get_config(args.model).family
    if family == "tovalix":
        run_tovalix(args, peaks, timer)
    elif family == "zikezen":
        run_zikezen(args, peaks, timer)
    elif family == "zigipel":
        run_zigipel(args, peaks, timer)
    else:
        run_roluzen(args, peaks, timer)


def run_tovalix(args, peaks, timer) -> None:
    from ..models.config import get_config
    from ..models.mixers import ForgetGateMemorySpec, RotaryAttentionSpec, TokenShiftMemorySpec
    from ..models.stack_exec import FEW_OUTPUTS, rope_table
    from . import functional as F
    from . import kernels as K
    from . import stack_kernels as SK
    report = reporter(args, peaks, timer)
    dev, bf = torch.device("cuda"), torch.bfloat16
    cfg = get_config(args.model)
    first = lambda t: next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, t))  # noqa: E731
    a, wk, fg, D = first(RotaryAttentionSpec), first(TokenShiftMemorySpec), first(ForgetGateMemorySpec), cfg.embed_dim
    rand = lambda *s: torch.randn(*s, device=dev).to(bf)  # noqa: E731
    for phase, rb, B, ctx in phases(args):
        n, one = rb.n, phase == "decode"
        # --- residual, norms, token shift
        x, y, w, h = torch.randn(n, 1, D, device=dev), rand(n, D), torch.ones(D, device=dev, dtype=bf), rand(n, D)
        unit, mu, last = torch.ones(1, device=dev, dtype=bf), rand(5, D), torch.zeros(B, D, device=dev)
        kw = dict(y=y, mix=unit, w_out=unit, w_in=unit, groups=cfg.norm_groups)
        report(f"stream_step_{phase}", lambda: SK.stream_step(x, 1e-6, norm_w=w, **kw), n * D * 12.0)
        report(f"stream_step_groups4_{phase}", lambda: SK.stream_step(x, 1e-6, norm_w=w, **{**kw, "groups": 4}), n * D * 12.0)
        report(f"stream_step_row_{phase}", lambda: SK.stream_step(x, 1e-6, raw=True, **kw), n * D * 12.0)
        report(f"stream_step_normed_{phase}", lambda: SK.stream_step(x, 1e-6, norm_w=w, wy=w, **kw), n * D * 12.0)
        if one:
            report("stream_step_shift_decode", lambda: SK.stream_step(x, 1e-6, norm_w=w, shift=(mu, last), rb=rb, **kw), n * D * 28.0)
        else:
            report("token_shift_prefill", lambda: SK.token_shift(h, mu, last, rb), n * D * 12.0)
        report(f"like_rmsnorm_{phase}", lambda: K.rmsnorm_fwd(y, w, 1e-6, want_rstd=False), n * D * 4.0)
        # --- per-layer token input
        N = cfg.token_side
        table, gw, z = rand(cfg.vocab_size, 4 * N), rand(N, D), torch.randn(n, N, device=dev)
        rows = dict(tokens=rb.tokens, rows=table, col=N)
        if one and N <= FEW_OUTPUTS:
            report("side_gate_decode", lambda: SK.few_outputs(h, gw, SK.ACT_GELU_ROW, **rows), n * D * 2.0 + N * D * 2)
            report("like_narrow_gemm_decode", lambda: K.gemm(h, gw), n * D * 2.0 + N * D * 2)
        else:
            report(f"small_act_{phase}", lambda: SK.small_act(z, bf, SK.ACT_GELU_ROW, **rows), n * N * 6.0)
        # --- feed-forward activation
        ff = cfg.hidden_dim
        up, act = rand(n, ff), rand(2)
        report(f"xielu_{phase}", lambda: SK.xielu_(up, act), n * ff * 4.0)
        half = rand(n, ff)
        report(f"like_glu_{phase}", lambda: K.glu_fwd(half, up, K.GLU_SILU), n * ff * 6.0)
        del up, half
        # --- matrix memories
        for name, sp, mode in (("wkv", wk, SK.GATES_BONUS), ("hgrn2", fg, SK.GATES_LOWER)):
            H, dk, dv = sp.heads, sp.dim, getattr(sp, "vdim", sp.dim)
            bonus = mode == SK.GATES_BONUS
            q, k, v, g = rand(n, H * dk), rand(n, H * dk) if bonus else None, rand(n, H * dv), rand(n, H * dv) if bonus else None
            z, c0, c1 = torch.randn(n, H * dk, device=dev), rand(H * dk) + (-3 if bonus else 2), torch.rand(H * dk, device=dev).to(bf)
            S, nw = torch.zeros(B, H, dk, dv, device=dev), torch.ones(H * dv if bonus else dv, device=dev, dtype=bf)
            nb = n * H * (dk * (6.0 + 2 * bonus) + dv * (4.0 + 2 * bonus)) + B * H * dk * dv * 8.0
            fl = 0.0 if one else n * H * (4.0 * dk * dv + 16 * (dk + dv))
            report(f"{name}_{phase}", lambda: SK.gated_linear(mode, q, k, v, z, c0, c1, rb, H, dk, dv, S, nw, 1e-6, gate=g,  # noqa: B023
                                                              per_head=bonus), nb, fl)
            del q, k, v, g, z, S
        # --- attention
        NQ, NK, NV = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
        kp, vp, table = page_pool(B, ctx, NK, NV)
        proj, q = rand(n, NQ + NK + NV), rand(n, NQ)
        cos, sin = rope_table(ctx, a.rot_dims, a.rot_base, dev)
        report(f"rope_norm_write_{phase}", lambda: SK.rope_norm_write(proj, 0, NQ, NQ + NK, cos, sin, a.rot_dims, 1e-6, rb, table, 64,
                                                                      a.heads, a.kv_heads, a.dim, a.vdim, kp, vp),
               n * (NQ + NK + NV) * 4.0)
        if one:
            keys = (ctx - 1) % a.chunk + 1
            nb = B * keys * (NK + NV) * 2.0 + n * NQ * 4.0
            split = K.decode_split_tokens(B, a.kv_heads, min(ctx, a.chunk + 128))
            dkw = dict(num_kv_heads=a.kv_heads, page_size=64, max_ctx=ctx, split_tokens=split, scale=a.scale)
            q3, lens_t = q.view(B, a.heads, a.dim), rb.pos0 + 1
            pd = lambda **o: K.paged_decode(q3, kp, vp, table, rb.slot, lens_t, **dkw, **o)  # noqa: E731
            report("attention_decode", lambda: pd(softcap=a.softcap, chunk=a.chunk), nb)
            report("like_paged_decode", lambda: pd(window=keys), nb, note="as many keys")
        else:
            full = sum(i % a.chunk + 1 for i in range(args.seq)) * float(B)
            fl, nb = full * a.heads * a.dim * 4.0, n * (2 * NQ + NK + NV) * 2.0
            pk = dict(num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, scale=a.scale)
            report("attention_prefill", lambda: K.attn_fwd_paged(q, kp, vp, rb, table, 64, softcap=a.softcap, chunk=a.chunk, **pk), nb, fl)
            report("attention_prefill_uncapped", lambda: K.attn_fwd_paged(q, kp, vp, rb, table, 64, chunk=a.chunk, **pk), nb, fl)
            q4 = q.view(B, args.seq, a.heads, a.dim)
            k4, v4 = (rand(B, args.seq, a.kv_heads, a.dim) for _ in range(2))
            seg = torch.ones(B, args.seq, dtype=torch.int32, device=dev)
            win = sum(min(i + 1, a.chunk) for i in range(args.seq)) * float(B) * a.heads * a.dim * 4.0
            att = lambda s: F.attention(q4, k4, v4, scale=a.scale, causal=True, window=a.chunk, seg_q=s, seg_k=s)  # noqa: E731
            with torch.no_grad():
                report("like_attn_fwd", lambda: att(None), nb, win, note="window as long as a chunk")
                report("like_attn_fwd_segments", lambda: att(seg), nb, win, note="as the padded prefill of uniform decoders calls it")


def run_zikezen(args, peaks, timer) -> None:
    from ..models.config import get_config
    from ..models.stack_exec import rope_table
    from . import functional as F
    from . import kernels as K
    from . import moe as uniform_moe
    from . import reference as R
    from . import stack_kernels as SK
    report = reporter(args, peaks, timer)
    dev, bf = torch.device("cuda"), torch.bfloat16
    cfg = get_config(args.model)
    sp = cfg.layer_specs[0].mixer
    ex = next(s for s in cfg.layer_specs if s.ff_kind == "experts")
    a, gl, D = sp.left, sp.right, cfg.embed_dim
    rand = lambda *s: torch.randn(*s, device=dev).to(bf)  # noqa: E731
    E, top, ff = ex.experts, ex.top, ex.ff
    gate_up, down, router, corr = rand(E, 2 * ff, D), rand(E, D, ff), rand(E, D), rand(E) * 0.01
    for phase, rb, B, ctx in phases(args):
        n, one = rb.n, phase == "decode"
        # --- residual
        x, y, w, h = torch.randn(n, 1, D, device=dev), rand(n, D), torch.ones(D, device=dev, dtype=bf), rand(n, D)
        unit, table, pos = torch.ones(1, device=dev, dtype=bf), rand(cfg.vocab_size, D), rand(cfg.positions, D)
        kw = dict(y=y, wy=w, mix=unit, w_out=unit, w_in=unit, norm_w=w)
        report(f"stream_step_normed_{phase}", lambda: SK.stream_step(x, 1e-6, **kw), n * D * 12.0)
        report(f"stream_step_again_{phase}", lambda: SK.stream_step(x, 1e-6, tokens=rb.tokens, embed=table, embed_scale=2.0, pos=pos, rb=rb,
                                                                    **kw), n * D * 14.0, note="tokens of one row")
        report(f"like_rmsnorm_{phase}", lambda: K.rmsnorm_fwd(y, w, 1e-6, want_rstd=False), n * D * 4.0)
        del x, table, pos
        # --- gated linear attention
        H, dk, dv, rank = gl.heads, gl.dim, gl.vdim, gl.decay_rank
        q, k, v, g = rand(n, H * dk), rand(n, H * dk), rand(n, H * dv), rand(n, H * dv)
        z, c0, xr, w2 = torch.randn(n, H * dk, device=dev), rand(H * dk) + 2, rand(n, rank), rand(H * dk, rank) * rank ** -0.5
        S, nw, nwh = torch.zeros(B, H, dk, dv, device=dev), torch.ones(dv, device=dev, dtype=bf), torch.ones(H * dv, device=dev, dtype=bf)
        nb, fl = n * H * (dk * 8.0 + dv * 6) + B * H * dk * dv * 8.0, 0.0 if one else n * H * (4.0 * dk * dv + 16 * (dk + dv))
        run_ = lambda mode, zz, kk, c1, **o: SK.gated_linear(mode, q, kk, v, zz, c0, c1, rb, H, dk, dv, S, o.pop("nw", nw), 1e-6, gate=g, **o)  # noqa: E731
        report(f"gla_{phase}", lambda: run_(SK.GATES_ROOT, z, k, None, q_scale=0.1, tau=16.0), nb, fl)
        if one:
            report("gla_bottleneck_decode", lambda: run_(SK.GATES_ROOT, None, k, None, q_scale=0.1, tau=16.0, low_rank=(xr, w2)),
                   nb - n * H * dk * 4.0 + n * rank * 2 + H * dk * rank * 2)
        report(f"like_wkv_{phase}", lambda: run_(SK.GATES_BONUS, z, k, c0, per_head=True, nw=nwh), nb, fl, note="same sizes")
        report(f"like_hgrn2_{phase}", lambda: run_(SK.GATES_LOWER, z, None, torch.sigmoid(c0)), nb - n * H * dk * 2, fl, note="same sizes")
        report(f"gates_product_{phase}", lambda: K.gemm(xr, w2, out_dtype=torch.float32), n * (rank * 2.0 + H * dk * 4) + H * dk * rank * 2)
        del q, k, v, g, z, S
        # --- attention
        NQ, NK = a.heads * a.dim, a.kv_heads * a.dim
        kp, vp, table = page_pool(B, ctx, NK, NK)
        proj, q, hw = rand(n, NQ + 2 * NK), rand(n, NQ), torch.ones(a.dim, device=dev, dtype=bf)
        cos, sin = rope_table(ctx, a.rot_dims, a.rot_base, dev)
        rope = lambda **o: SK.rope_norm_write(proj, 0, NQ, NQ + NK, cos, sin, a.rot_dims, 1e-6, rb, table, 64, a.heads, a.kv_heads, a.dim, a.vdim,  # noqa: E731
                                              kp, vp, **o)
        report(f"rope_norm_write_{phase}", lambda: rope(q_w=hw, k_w=hw, interleaved=True), n * (NQ + 2 * NK) * 4.0)
        report(f"like_rope_norm_write_{phase}", lambda: rope(), n * (NQ + 2 * NK) * 4.0, note="halves, no weights")
        if one:
            keys = min(ctx, a.window)
            nb = B * keys * 2 * NK * 2.0 + n * NQ * 4.0
            split = K.decode_split_tokens(B, a.kv_heads, min(ctx, a.window + 128))
            q3, lens_t = q.view(B, a.heads, a.dim), rb.pos0 + 1
            pd = lambda **o: K.paged_decode(q3, kp, vp, table, rb.slot, lens_t, num_kv_heads=a.kv_heads, page_size=64, max_ctx=ctx,  # noqa: E731
                                            split_tokens=split, scale=a.scale, window=a.window, **o)
            report("attention_decode", lambda: pd(sink=0.0, out_scale=0.7), nb)
            report("like_paged_decode", lambda: pd(), nb, note="no sink")
        else:
            fl = sum(min(i + 1, a.window) for i in range(args.seq)) * float(B) * a.heads * a.dim * 4.0
            nb = n * (2 * NQ + 2 * NK) * 2.0
            pk = dict(num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, scale=a.scale, window=a.window)
            report("attention_prefill", lambda: K.attn_fwd_paged(q, kp, vp, rb, table, 64, sink=0.0, out_scale=0.7, **pk), nb, fl)
            q4 = q.view(B, args.seq, a.heads, a.dim)
            k4, v4 = (rand(B, args.seq, a.kv_heads, a.dim) for _ in range(2))
            seg = torch.ones(B, args.seq, dtype=torch.int32, device=dev)
            att = lambda s: F.attention(q4, k4, v4, scale=a.scale, causal=True, window=a.window, seg_q=s, seg_k=s)  # noqa: E731
            with torch.no_grad():
                report("like_attn_fwd", lambda: att(None), nb, fl, note="same window")
                report("like_attn_fwd_segments", lambda: att(seg), nb, fl, note="as the padded prefill of uniform decoders calls it")
            del q4, k4, v4
        del kp, vp, proj, q
        # --- experts
        logits = torch.randn(n, E, device=dev)
        used = (torch.softmax(logits, -1) + corr).topk(top, -1).indices.unique().numel()
        nb, fl = n * D * 4.0 + used * 6.0 * ff * D + n * E * 4, n * top * 6.0 * ff * D
        report(f"router_{phase}", (lambda: SK.few_outputs(h, router)) if one else (lambda: K.gemm(h, router, out_dtype=torch.float32)),
               n * (D * 2.0 + E * 4) + E * D * 2)
        report(f"experts_{phase}", lambda: SK.moe(h, logits, corr, gate_up, down, top, rb), nb, fl)
        gw, uw = gate_up[:, :ff].contiguous(), gate_up[:, ff:].contiguous()

        def uniform():
            wts, idx, _ = R.topk_router_ref(logits, top, True)
            return uniform_moe.experts(h, wts, idx, gw, uw, down)
        with torch.no_grad():
            report(f"like_experts_{phase}", uniform, nb, fl, note="expert layer of uniform decoders, routing included")
        half, up = rand(n, cfg.hidden_dim), rand(n, cfg.hidden_dim)
        report(f"glu_{phase}", lambda: K.glu_fwd(half, up, K.GLU_SILU), n * cfg.hidden_dim * 6.0)
        del half, up, gw, uw


def run_zigipel(args, peaks, timer) -> None:
    from ..models.config import get_config
    from ..models.mixers import DistanceAttention, DistanceAttentionSpec, LatentAttention, LatentAttentionSpec
    from ..models.stack_exec import rope_table
    from . import functional as F
    from . import kernels as K
    from . import stack_kernels as SK
    report = reporter(args, peaks, timer)
    dev, bf = torch.device("cuda"), torch.bfloat16
    cfg = get_config(args.model)
    first = lambda t: next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, t))  # noqa: E731
    a, la, D, ff = first(DistanceAttentionSpec), first(LatentAttentionSpec), cfg.embed_dim, cfg.hidden_dim
    rand = lambda *s: torch.randn(*s, device=dev).to(bf)  # noqa: E731
    for phase, rb, B, ctx in phases(args):
        n, one = rb.n, phase == "decode"
        # --- residual, embedding, token shift
        x, y, w, h = torch.randn(n, 1, D, device=dev), rand(n, D), torch.ones(D, device=dev, dtype=bf), rand(n, D)
        unit, mu, before = torch.ones(1, device=dev, dtype=bf), rand(1, D), torch.zeros(B, D, device=dev)
        table, pairs, last = rand(cfg.vocab_size, D), rand(cfg.bigram[0] + 1, D), torch.zeros(B, dtype=torch.int64, device=dev)
        ids = torch.randint(0, cfg.vocab_size, (n,), device=dev)
        kw = dict(y=y, mix=unit, w_out=unit, w_in=unit, norm_w=w)
        if one:
            report("stream_step_shift_decode", lambda: SK.stream_step(x, 1e-6, shift=(mu, before), both=True, rb=rb, **kw), n * D * 22.0)
        else:
            report("stream_step_prefill", lambda: SK.stream_step(x, 1e-6, **kw), n * D * 12.0)
            report("token_shift_prefill", lambda: SK.token_shift(h, mu, before, rb), n * D * 4.0)
        row = torch.empty(n, 2 * D, device=dev, dtype=bf)
        report(f"embedding_{phase}", lambda: SK.stream_step(x, 1e-6, tokens=ids, embed=table, pairs=(pairs, cfg.bigram, last), rb=rb,
                                                            start_out=row[:, D:], w_in=unit, norm_w=w), n * D * 12.0)
        win = rand(D, 2 * D)
        report(f"loop_product_{phase}", lambda: K.gemm(row, win, out=x.view(n, D), bias=y[0]), n * D * 8.0 + 4.0 * D * D, 4.0 * n * D * D)
        report(f"like_rmsnorm_{phase}", lambda: K.rmsnorm_fwd(y, w, 1e-6, want_rstd=False), n * D * 4.0)
        half, up, wide_row = rand(n, ff), rand(n, ff), torch.empty(n, ff + a.heads * a.vdim, device=dev, dtype=bf)
        report(f"glu_gelu_{phase}", lambda: K.glu_fwd(half, up, K.GLU_GELU, wide_row[:, a.heads * a.vdim:]), n * ff * 6.0)
        report(f"like_glu_{phase}", lambda: K.glu_fwd(half, up, K.GLU_SILU), n * ff * 6.0)
        del x, table, pairs, half, up, wide_row, row, win
        # --- distance attention
        m = DistanceAttention(a, 8, 1e-6, bf, dev)
        NQ, NK, NV = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
        kp, vp, pt = page_pool(B, ctx, NK, NV)
        proj, gate, sinks, bias = rand(n, NQ + NK + NV), rand(n, a.heads), torch.zeros(a.heads, device=dev), m.bias_table(ctx)
        report(f"value_norm_write_{phase}", lambda: SK.rope_norm_write(proj, 0, NQ, NQ + NK, None, None, 0, 1e-6, rb, pt, 64, 0, a.kv_heads,
                                                                       a.dim, a.vdim, kp, vp, norm_qk=False, norm_v=True), n * (NK + NV) * 4.0)
        cos, sin = rope_table(ctx, a.dim, 1e4, dev)
        report(f"like_rope_norm_write_{phase}", lambda: SK.rope_norm_write(proj, 0, NQ, NQ + NK, cos, sin, a.dim, 1e-6, rb, pt, 64, a.heads,
                                                                           a.kv_heads, a.dim, a.vdim, kp, vp), n * (NQ + NK + NV) * 4.0)
        seen = sum(min(i + 1, a.window) + min(max(i + 1 - a.window, 0), a.keep_first) for i in range(args.seq)) * float(B)
        ext = dict(keep_first=a.keep_first, bias=bias, sinks=sinks, gate=gate)
        if one:
            keys = min(ctx, a.window + a.keep_first)
            nb = B * keys * (NK + NV) * 2.0 + n * NQ * 4.0
            split = K.decode_split_tokens(B, a.kv_heads, min(ctx, a.window + a.keep_first + 128))
            q3, lens_t = proj[:, :NQ].unflatten(1, (a.heads, a.dim)), rb.pos0 + 1
            pd = lambda **o: K.paged_decode(q3, kp, vp, pt, rb.slot, lens_t, num_kv_heads=a.kv_heads, page_size=64, max_ctx=ctx,  # noqa: E731
                                            split_tokens=split, scale=a.scale, window=a.window, **o)
            report("attention_decode", lambda: pd(**ext), nb)
            report("like_paged_decode", lambda: pd(), nb, note="same window; no bias, sinks, gates, kept tokens")
        else:
            nb, fl = n * (2 * NQ + NK + NV) * 2.0, seen * a.heads * (a.dim + a.vdim) * 2.0
            pk = dict(num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, scale=a.scale, window=a.window)
            q3 = proj.as_strided((n, a.heads, a.dim), (proj.stride(0), a.dim, 1))
            report("attention_prefill", lambda: K.attn_fwd_paged(q3, kp, vp, rb, pt, 64, **ext, **pk), nb, fl)
            q4 = rand(B, args.seq, a.heads, a.dim)
            k4, v4 = (rand(B, args.seq, a.kv_heads, a.dim) for _ in range(2))
            seg = torch.ones(B, args.seq, dtype=torch.int32, device=dev)
            win = sum(min(i + 1, a.window) for i in range(args.seq)) * float(B) * a.heads * a.dim * 4.0
            att = lambda s: F.attention(q4, k4, v4, scale=a.scale, causal=True, window=a.window, seg_q=s, seg_k=s)  # noqa: E731
            with torch.no_grad():
                report("like_attn_fwd", lambda: att(None), nb, win, note="same window, no bias")
                report("like_attn_fwd_segments", lambda: att(seg), nb, win, note="as the padded prefill of uniform decoders calls it")
            del q4, k4, v4
        del kp, vp, proj
        # --- latent attention
        m = LatentAttention(la, D, 1e-6, bf, dev)
        for p in m.parameters():
            p.data.normal_(0, 0.05)
        H, R, qd, W = la.heads, la.kv_rank, la.dim + la.rot_dim, la.stored(bf)[0]
        wide, wide_v = la.tile_heads()
        pages = -(-ctx // 64)
        pool = torch.randn(B * pages, 64, W, device=dev).to(bf)
        pool[..., la.width:] = 0
        pt = torch.randperm(B * pages, device=dev).int().view(B, pages)
        proj, cos_sin = rand(n, H * qd + la.width), rope_table(ctx, la.rot_dims, la.rot_base, dev, la.rot_scaling)
        report(f"latent_write_{phase}", lambda: SK.latent_write(proj, H * qd, m.kv_norm.weight, *cos_sin, la.rot_dims, 1e-6, rb, pt, 64, H, la.dim,
                                                                la.rot_dim, R, pool), n * (H * la.rot_dim * 4.0 + la.width * 4.0))
        sinks, q = torch.zeros(H, device=dev), proj[:, :H * qd].unflatten(1, (H, qd))
        if one:
            uk, uv = m.uk_proj.weight.data.view(H, la.dim, R), m.uv_proj.weight.data.view(H, la.vdim, R)
            q1, out = torch.zeros(n, H, W, device=dev, dtype=bf), torch.empty(n, H, la.vdim, device=dev, dtype=bf)
            report("head_product_keys_decode", lambda: SK.head_product(q, uk, q1, tail=la.rot_dim), n * H * (qd + W) * 2.0 + uk.numel() * 2,
                   2.0 * n * H * la.dim * R)
            dec = lambda: SK.latent_decode(q1, pool, pt, 64, rb.slot, rb.pos0 + 1, rank=R, scale=la.scale, window=la.window, sinks=sinks,  # noqa: E731
                                           max_ctx=ctx)
            keys = min(ctx, la.window)
            report("latent_decode", dec, B * keys * la.width * 2.0 + n * H * (la.width + R) * 2.0, 2.0 * B * keys * H * (la.width + R))
            att = dec()
            report("head_product_values_decode", lambda: SK.head_product(att, uv, out, transposed=True), n * H * (R + la.vdim) * 2.0 + uv.numel() * 2,
                   2.0 * n * H * la.vdim * R)
            wk = rand(H * la.dim, D)
            report("like_narrow_gemm_decode", lambda: K.gemm(h, wk), n * D * 2.0 + n * H * la.dim * 2 + wk.numel() * 2, note="a projection")
        else:
            plan, expand = rb.latent_plan(la.window), m.expansion(W)
            rows = plan.blocks[0].shape[0] * 64
            report("latent_gather_prefill", lambda: SK.latent_gather(pool, *plan.blocks, pt, 64), rows * W * 4.0)
            g = SK.latent_gather(pool, *plan.blocks, pt, 64)
            gk, keys = g[:, :expand.shape[1]], H * (la.dim if la.split_keys else wide)
            report("latent_expand_prefill", lambda: K.gemm(gk, expand), rows * (R + H * (la.dim + la.vdim)) * 2.0,
                   2.0 * rows * R * H * (la.dim + la.vdim))
            kv = K.gemm(gk, expand)
            q3 = proj.as_strided((n, H, wide), (proj.stride(0), qd, 1))
            fl = sum(min(i + 1, la.window) for i in range(args.seq)) * float(B) * H * (qd + la.vdim) * 2.0
            report("latent_attention_prefill", lambda: K.attn_fwd_paged(q3, kv[:, :keys], kv[:, keys:], rb, plan.table, 64, num_heads=H,
                                                                        num_kv_heads=H, head_dim=wide, scale=la.scale, window=la.window,
                                                                        sinks=sinks, value_dim=la.vdim, tiles=plan.tiles, slots=plan.entries,
                                                                        shared_keys=(g, R) if la.split_keys else None),
                   n * H * (2.0 * qd + 2.0 * la.vdim) * 2.0, fl)
        del pool, proj


def run_roluzen(args, peaks, timer) -> None:
    from ..models.config import get_config
    from ..models.mixers import ParallelSpec, RGLRUMixer, RGLRUSpec
    from . import functional as F
    from . import kernels as K
    from . import stack_kernels as SK
    report = reporter(args, peaks, timer)
    dev, bf = torch.device("cuda"), torch.bfloat16
    cfg = get_config(args.model)
    par = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, ParallelSpec))
    rec = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, RGLRUSpec))
    a, mm, D, S = par.left, par.right, cfg.embed_dim, max(cfg.streams, 1)
    bias = torch.randn(a.heads, a.bias_max + 1, device=dev)
    aw = dict(scale=a.scale, window=a.window)
    for phase, rb, B, ctx in phases(args):
        n, one = rb.n, phase == "decode"
        # --- streams
        x = torch.randn(n, S, D, device=dev)
        y, y2 = (torch.randn(n, D, device=dev).to(bf) for _ in range(2))
        w = torch.ones(D, device=dev, dtype=bf)
        mix, vec = torch.eye(S, device=dev, dtype=bf), torch.ones(S, device=dev, dtype=bf)
        kw = dict(mix=mix, w_out=vec, w_in=vec, norm_w=w)
        report(f"stream_step_{phase}", lambda: SK.stream_step(x, 1e-6, y=y, **kw), n * D * (8.0 * S + 4))
        report(f"stream_step_pair_{phase}", lambda: SK.stream_step(x, 1e-6, y=y, y2=y2, wy=w, wy2=w, **kw), n * D * (8.0 * S + 6))
        report(f"like_rmsnorm_{phase}", lambda: K.rmsnorm_fwd(y, w, 1e-6, want_rstd=False), n * D * 4.0)
        del x
        # --- gated recurrence
        W, bs = rec.width, rec.width // rec.blocks
        m = RGLRUMixer(rec, 64, 1e-6, bf, dev)
        for p in m.parameters():
            p.data.normal_(0, 0.05)
        st = {k: torch.zeros(B, *s, device=dev) for k, s in rec.state_shapes().items()}
        proj = torch.randn(n, 2 * W, device=dev).to(bf)
        wbytes = 2.0 * rec.blocks * bs * bs * 2
        report(f"rglru_{phase}", lambda: SK.rglru(proj, W, 0, m, rb, st), n * W * 6.0 + wbytes + B * W * (8 + 4.0 * rec.conv),
               n * W * bs * 4.0)
        del proj
        # --- matrix memory
        H, dk, dv = mm.heads, mm.dim, mm.vdim
        st = {k: torch.zeros(B, *s, device=dev) for k, s in mm.state_shapes().items()}
        proj = torch.randn(n, H * (2 * dk + dv), device=dev).to(bf)
        gates = torch.randn(n, 2 * H, device=dev)
        b = torch.zeros(H, device=dev, dtype=bf)
        chunk = 1 if one else 64
        fl = n * H * (4.0 * dk * dv + chunk * (dk + dv))
        report(f"mlstm_{phase}", lambda: SK.mlstm(proj, 0, H * dk, 2 * H * dk, gates, b, b, mm.gate_cap, rb, H, dk, dv, st),
               n * H * (4.0 * dk + 2 * dv + 4 * dv) + B * H * dk * dv * 8.0, 0.0 if one else fl)
        del proj
        # --- attention
        NQ, NK, NV = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
        kp, vp, table = page_pool(B, ctx, NK, NV)
        proj = torch.randn(n, NQ + NK + NV, device=dev).to(bf)
        qw, kwt = torch.ones(NQ, device=dev, dtype=bf), torch.ones(NK, device=dev, dtype=bf)
        report(f"qk_norm_write_{phase}", lambda: SK.qk_norm_write(proj, 0, NQ, NQ + NK, qw, kwt, 1e-6, rb, table, 64, kp, vp, NQ),
               n * (NQ + NK + NV) * 4.0)
        q = torch.randn(n, NQ, device=dev).to(bf)
        if one:
            keys = min(ctx, a.window + a.keep_first)
            nb = B * keys * (NK + NV) * 2.0 + n * NQ * 4.0
            split = K.decode_split_tokens(B, a.kv_heads, min(ctx, a.window + a.keep_first + 128))
            dkw = dict(num_kv_heads=a.kv_heads, page_size=64, max_ctx=ctx, split_tokens=split, **aw)
            q3 = q.view(B, a.heads, a.dim)
            lens_t, slots = rb.pos0 + 1, rb.slot
            report("attention_decode", lambda: K.paged_decode(q3, kp, vp, table, slots, lens_t, keep_first=a.keep_first, bias=bias, **dkw), nb)
            report("like_paged_decode", lambda: K.paged_decode(q3, kp, vp, table, slots, lens_t, **dkw), nb, note="same window, no bias")
        else:
            full = sum(min(i + 1, a.window) for i in range(args.seq)) * float(B)
            fl, nb = full * a.heads * a.dim * 4.0, n * (2 * NQ + NK + NV) * 2.0
            report("attention_prefill", lambda: K.attn_fwd_paged(q, kp, vp, rb, table, 64, num_heads=a.heads, num_kv_heads=a.kv_heads,
                                                                 head_dim=a.dim, keep_first=a.keep_first, bias=bias, **aw), nb, fl)
            q4 = q.view(B, args.seq, a.heads, a.dim)
            k4, v4 = (torch.randn(B, args.seq, a.kv_heads, a.dim, device=dev).to(bf) for _ in range(2))
            seg = torch.ones(B, args.seq, dtype=torch.int32, device=dev)
            att = lambda s: F.attention(q4, k4, v4, scale=a.scale, causal=True, window=a.window, seg_q=s, seg_k=s)  # noqa: E731
            with torch.no_grad():
                report("like_attn_fwd", lambda: att(None), nb, fl, note="same window, no bias")
                report("like_attn_fwd_segments", lambda: att(seg), nb, fl, note="as the padded prefill of uniform decoders calls it")
        # --- output gates
        C1, C2 = a.heads * a.vdim, H * dv
        g = torch.randn(n, C1 + C2, device=dev).to(bf)
        att_o, o = torch.randn(n, C1, device=dev).to(bf), torch.randn(n, H, dv, device=dev)
        nw = torch.ones(C2, device=dev, dtype=bf)
        report(f"gate_outputs_{phase}", lambda: SK.gate_outputs(att_o, o, g, 0, C1, nw, 1e-6, H, dv), n * (C1 * 6.0 + C2 * 8.0))
        if one:
            h, gw = torch.randn(n, D, device=dev).to(bf), torch.randn(2 * H, D, device=dev).to(bf)
            report("few_outputs_decode", lambda: SK.few_outputs(h, gw), n * D * 2.0 + 4.0 * H * D)
