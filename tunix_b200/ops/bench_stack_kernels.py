"""Micro-benchmarks of the layer-stack kernels: `python -m tunix_b200.ops.bench_kernels stack [--model roluzen_8b]
[--batch 4 --seq 4096] [--decode-batch 64 --decode-ctx 1024] [--only mlstm_prefill,...]`.

One JSON line per kernel at the sizes of a preset: median time with L2 flushed between iterations, the algorithmic bytes and
operations (every input read once, every output written once; no repeated or split work counted), and the fraction of the
roofline, i.e. the larger of bytes / copy bandwidth and operations / GEMM throughput over the measured time. The like kernels
of uniform decoders (flash attention with the same window as a prefill calls it, paged decode, RMS norm) come beside them."""
from __future__ import annotations

import json

import torch


def run(args, peaks, timer) -> None:
    from ..models.config import get_config
    from ..models.mixers import MatrixMemory, ParallelSpec, RGLRUMixer, RGLRUSpec
    from . import functional as F
    from . import kernels as K
    from . import stack_kernels as SK
    from .ragged import RaggedBatch
    peak_tf, peak_gb, which = peaks
    dev, bf = torch.device("cuda"), torch.bfloat16
    cfg = get_config(args.model)
    par = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, ParallelSpec))
    rec = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, RGLRUSpec))
    a, mm, D, S = par.left, par.right, cfg.embed_dim, max(cfg.streams, 1)
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

    def pool(B, ctx):
        pages = -(-ctx // 64)
        mk = lambda n: torch.randn(B * pages, 64, n, device=dev).to(bf)  # noqa: E731
        return mk(a.kv_heads * a.dim), mk(a.kv_heads * a.vdim), torch.randperm(B * pages, device=dev).int().view(B, pages)

    bias = torch.randn(a.heads, a.bias_max + 1, device=dev)
    aw = dict(scale=a.scale, window=a.window)
    lens = {"prefill": [args.seq] * args.batch, "decode": [1] * args.decode_batch}
    for phase, ls in lens.items():
        B, n, one = len(ls), sum(ls), phase == "decode"
        ctx = args.decode_ctx if one else args.seq
        rb = RaggedBatch.build([(i, ctx - 1 if one else 0, [1] * L) for i, L in enumerate(ls)], dev)
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
        kp, vp, table = pool(B, ctx)
        NQ, NK, NV = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
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
