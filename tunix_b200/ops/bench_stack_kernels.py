"""Micro-benchmarks of the layer-stack kernels: `python -m tunix_b200.ops.bench_kernels stack [--model roluzen_8b|tovalix_8b|zikezen_8b]
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
