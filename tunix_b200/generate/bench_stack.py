"""Serving throughput of layer-stack models beside the closest uniform decoder of equal size:
`python bench.py --workload stack_serving` or
`python -m tunix_b200.generate.bench_stack [--models roluzen_2b,roluzen_8b,tovalix_2b,..,zigipel_2b,zigipel_8b]`.

For every size: prefill tokens/s (`--prefill-seqs` prompts of `--prefill-len` tokens, one sampled token each) and decode
tokens/s (`--decode-seqs` sequences at context `--decode-ctx`, `--decode-steps` captured steps), both through
`PagedEngine.__call__`, random-init weights, uniform random token ids. The other model has the same width, feed-forward
(of equal size where only one of them is gated, as much as a token passes where there are experts), attention heads, vocabulary and number of layer passes, with
sliding-window attention in every layer, of the same window or as long as the chunks. Models with experts stand beside a second
one, whose feed-forwards are all such experts.
Times are CUDA events around the call after a warm-up call; a decode step streams the weights (far more than L2), the
prefill's activations exceed L2 too."""
from __future__ import annotations

import argparse
import json
import sys

import numpy as np
import torch


class _Ids:
    def encode(self, s):
        return [3]

    def decode(self, ids):
        return ""

    def bos_id(self):
        return 1

    def eos_id(self):
        return -1

    def pad_id(self):
        return 0


def closest_config(cfg):
    """Uniform decoder with the sizes of a layer-stack config: one attention + MLP layer per layer pass."""
    from ..models.config import ModelConfig
    att = next(a for a in (getattr(s.mixer, "left", s.mixer) for s in cfg.layer_specs) if hasattr(a, "kv_heads"))
    gated = all(s.ff_kind == "glu" for s in cfg.layer_specs)
    return ModelConfig(family="qwen3", num_layers=len(cfg.runs()), vocab_size=cfg.vocab_size, embed_dim=cfg.embed_dim,
                       hidden_dim=cfg.hidden_dim if gated else round(cfg.hidden_dim * 2 / 3 / 128) * 128, num_heads=att.heads,
                       head_dim=att.dim, num_kv_heads=att.kv_heads, qk_norm=True, sliding_window=att.window or att.chunk,
                       layer_pattern=("local",), dtype=torch.bfloat16)


def closest_experts_config(cfg):
    """The same with the experts of `cfg` in every layer, or None."""
    ex = next((s for s in cfg.layer_specs if s.ff_kind == "experts"), None)
    if ex is None:
        return None
    return closest_config(cfg).replace(num_experts=ex.experts, num_experts_per_tok=ex.top, moe_hidden_dim=ex.ff)


def flops_per_token(model) -> float:
    """2 x the weights of the projections a token passes (each layer pass and the experts it takes counted), head excluded."""
    cfg = model.config
    runs = cfg.runs() if hasattr(cfg, "runs") else range(cfg.num_layers)

    def weights(i):
        total = 0.0
        for p in model.layers[i].parameters():
            if p.dim() == 3:            # stacked experts
                top = cfg.layer_specs[i].top if hasattr(cfg, "layer_specs") else cfg.num_experts_per_tok
                total += p.numel() * (top / p.shape[0] if top else 1.0)
            elif p.dim() == 2:
                total += p.numel()
        return total
    loop_in = getattr(model, "loop_in", None)
    starts = 0 if loop_in is None else len(cfg.loop_starts()) * loop_in.weight.numel()
    return 2.0 * (sum(weights(i) for i in runs) + starts)


def measure(cfg, args) -> dict:
    from .. import _lib
    from ..common.configs import CacheConfig
    from ..models.transformer import create_model
    from ..ops import kernels as K
    from .engine import PagedEngine
    dev = torch.device("cuda")
    cfg = cfg.replace(dtype=torch.bfloat16, max_position=max(args.prefill_len, args.decode_ctx + args.decode_steps) + 64)
    model = create_model(cfg, device=dev, seed=0)
    rng = np.random.default_rng(0)

    def timed(eng, prompts, plen, steps):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        eng(prompt_token_ids=prompts, max_generation_steps=steps, max_prompt_length=plen, temperature=0.0, eos_tokens=[-1])
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1)

    def engine(seqs, total):
        return PagedEngine(model, _Ids(), CacheConfig(total, cfg.num_layers, cfg.num_kv_heads, cfg.head_dim), page_size=64,
                           max_running_requests=seqs, check_every=10 ** 9, prefix_caching=False)

    l0 = K.launch_count
    total = args.prefill_len + 64
    eng = engine(args.prefill_seqs, total)
    prompts = rng.integers(3, cfg.vocab_size, (args.prefill_seqs, args.prefill_len)).tolist()
    for _ in range(2):
        timed(eng, prompts, args.prefill_len, 1)
    pre = min(timed(eng, prompts, args.prefill_len, 1) for _ in range(args.repeats))
    del eng
    total = args.decode_ctx + args.decode_steps + 64
    eng = engine(args.decode_seqs, total)
    prompts = rng.integers(3, cfg.vocab_size, (args.decode_seqs, args.decode_ctx)).tolist()
    short, long = 5, 5 + args.decode_steps
    timed(eng, prompts, args.decode_ctx, long)
    a = b = float("inf")                # alternating, so that a change of clocks reaches both
    for _ in range(args.repeats):
        a = min(a, timed(eng, prompts, args.decode_ctx, short))
        b = min(b, timed(eng, prompts, args.decode_ctx, long))
    _lib.raise_if_kernel_error()
    step = (b - a) / args.decode_steps
    n_pre = args.prefill_seqs * args.prefill_len
    out = {"params": sum(p.numel() for p in model.parameters()), "layer_passes": len(cfg.runs()) if hasattr(cfg, "runs") else cfg.num_layers,
           "prefill_ms": pre, "prefill_tokens_per_sec": n_pre / pre * 1e3, "prefill_gemm_tflops": flops_per_token(model) * n_pre / pre / 1e9,
           "decode_ms_per_step": step, "decode_tokens_per_sec": args.decode_seqs / step * 1e3,
           "native_launches_outside_graph": K.launch_count - l0}
    if eng.pool.state is not None:
        out["state_bytes_per_sequence"] = eng.pool.state.nbytes_per_slot()
    del eng, model
    torch.cuda.empty_cache()
    return out


def add_arguments(ap) -> None:
    ap.add_argument("--models", default="roluzen_2b,roluzen_8b,tovalix_2b,tovalix_8b,zikezen_2b,zikezen_8b,zigipel_2b,zigipel_8b",
                    help="layer-stack presets (stack_serving)")
    ap.add_argument("--prefill-seqs", type=int, default=4)
    ap.add_argument("--prefill-len", type=int, default=4096)
    ap.add_argument("--decode-seqs", type=int, default=64)
    ap.add_argument("--decode-ctx", type=int, default=1024)
    ap.add_argument("--decode-steps", type=int, default=64)
    ap.add_argument("--repeats", type=int, default=3)


def run(args) -> int:
    from ..models.config import get_config
    for name in args.models.split(","):
        cfg = get_config(name)
        ours = measure(cfg, args)
        near, experts = measure(closest_config(cfg), args), closest_experts_config(cfg)
        print(json.dumps({"metric": "stack_serving", "model": name, "unit": "tokens/s", "value": ours["prefill_tokens_per_sec"],
                          "higher_is_better": True, "dtype": "bf16", "data": "synthetic uniform token ids, random-init weights",
                          "prefill": f"{args.prefill_seqs} x {args.prefill_len}",
                          "decode": f"{args.decode_seqs} sequences at context {args.decode_ctx}, {args.decode_steps} steps",
                          "stack": ours, "closest_uniform_decoder": near,
                          **({} if experts is None else {"closest_with_experts": measure(experts, args)})}), flush=True)
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    add_arguments(ap)
    return run(ap.parse_args(argv))


if __name__ == "__main__":
    sys.exit(main())
