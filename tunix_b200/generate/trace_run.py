"""Replays a trace of token ids through a model, step by step, and writes the logits that the trace asks for:

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every line of standard input is a step: {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [1]}], "end": []}.
Its entries run as one batch, from the cache and state that earlier steps left (`generate.engine.StepSession`); the logits
at the wanted places go to DIR/<step>.f32 as little-endian fp32 rows, then "done <step>" is printed. `--max-tokens` sizes
the page pool (64 tokens a page); four requests may be live at a time. Nothing is sampled."""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE, SLOTS = 64, 4


class _Ids:
    """The engine asks its tokenizer for the padding id only."""

    def pad_id(self):
        return 0

    def eos_id(self):
        return -1

    def bos_id(self):
        return None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits, one <step>.f32 per step that wants some")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time, each "
                    "request's count rounded up to whole pages")
    args = ap.parse_args(argv)
    import torch

    from ..common.configs import CacheConfig
    from ..models.automodel import AutoModel, ModelSource
    from ..models.hf_config import config_from_hf
    from .engine import PagedEngine, StepSession
    if not torch.cuda.is_available():
        raise RuntimeError("trace_run needs a CUDA device")
    dev = torch.device("cuda", 0)
    dtype = getattr(torch, args.dtype)
    cfg = config_from_hf(args.model, dtype=dtype)
    model, _ = AutoModel.from_pretrained(args.model, model_source=ModelSource.LOCAL, model_path=args.model, config=cfg, device=dev)
    pages = -(-args.max_tokens // PAGE)
    engine = PagedEngine(model, _Ids(), CacheConfig(pages * PAGE, cfg.num_layers, cfg.num_kv_heads, cfg.head_dim), page_size=PAGE,
                         max_running_requests=SLOTS, num_pages=pages)
    session = StepSession(engine)
    from .. import _lib
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = session.step([(e["id"], e["tokens"], e.get("want", ())) for e in step["entries"]], step.get("end", ()))
        if logits.shape[0]:
            data = logits.float().cpu().numpy().astype("<f4", copy=False).tobytes()
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                f.write(data)
        else:
            torch.cuda.synchronize()
        _lib.raise_if_kernel_error(dev)
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
