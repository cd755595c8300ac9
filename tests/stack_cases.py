"""Small Roluzen checkpoints with random weights for the layer-stack tests (config.json dict + tensors by name)."""
import json
import os

import torch


def attention(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.3, bias_max=40, size=20, keep_first=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max,
            "mask": {"size": size, "keep_first": keep_first}}


def memory(heads=2, dim=24, vdim=40, gate_cap=9.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}


def parallel(left=None, right=None, ff=72):
    return {"type": "parallel", "mixer": {"left": left or attention(), "right": right or memory()},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def rglru(width=80, blocks=5, conv=4, ff=56):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=48, vocab=101, streams=3, loop=None, eps=1e-5):
    return {"architecture": "Roluzen", "layers": layers, "loop": loop, "norm": {"eps": eps}, "streams": streams, "vocab": vocab,
            "width": width}


# sizes apart from each other, layers with and without feed-forward, loops and none, one stream and several, odd widths;
# "wide" has the head sizes and widths of the tensor-core kernels
CASES = {
    "mixed": config([rglru(), parallel(), parallel(ff=None), rglru(conv=2, ff=None)], loop={"start": 1, "stop": 3, "times": 2}),
    "one_stream": config([parallel(attention(heads=3, kv_heads=3, dim=8, vdim=8, keep_first=0, size=9), memory(3, 16, 8)), rglru(64, 1, 1)],
                         streams=1, width=40),
    "odd": config([parallel(attention(heads=2, kv_heads=1, dim=10, vdim=6, size=33, keep_first=70, bias_max=100), memory(1, 12, 33)),
                   rglru(36, 3, 3, ff=31)], width=36, streams=2, vocab=67, eps=1e-3),
    "wide": config([parallel(attention(heads=6, kv_heads=3, dim=64, vdim=64, scale=0.11, size=70, keep_first=5, bias_max=90),
                             memory(2, 40, 72), ff=128), rglru(128, 2, 4, ff=96)], width=128, streams=4, vocab=300,
                   loop={"start": 0, "stop": 1, "times": 3}),
}


def weights(cfg, seed=0, buckets=11):
    """Random tensors of the checkpoint, in bf16-representable fp32. Decays reach from fast to very slow and the bias table
    is large, so that far tokens, window edges and kept tokens matter."""
    g = torch.Generator().manual_seed(seed)
    w = {}

    def put(name, *shape, std=None, mean=0.0):
        std = (shape[-1] ** -0.5 if len(shape) > 1 else 0.2) if std is None else std
        w[name] = (mean + std * torch.randn(*shape, generator=g)).to(torch.bfloat16).float()

    D, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    put("embed", V, D, std=1.0)
    put("head", V, D)
    put("final.norm", D, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        put(p + "norm1", D, mean=1.0)
        if layer["type"] == "rglru":
            W, nb = m["width"], m["blocks"]
            for n in ("y", "x"):
                put(f"{p}mix.{n}", W, D)
                put(f"{p}mix.{n}.b", W)
            put(p + "mix.conv", W, m["conv"], std=0.6)
            put(p + "mix.conv.b", W)
            for n in ("ra", "ri"):
                put(f"{p}mix.{n}", nb, W // nb, W // nb)
                put(f"{p}mix.{n}.b", nb, W // nb)
            put(p + "mix.lam", W, std=2.0, mean=-3.0)
            put(p + "mix.o", D, W)
        else:
            a, r = m["left"], m["right"]
            H, G = a["heads"], a["kv_heads"]
            for n, rows in (("q", H * a["dim"]), ("k", G * a["dim"]), ("v", G * a["vdim"]), ("g", H * a["vdim"])):
                put(f"{p}mix.left.{n}", rows, D)
            put(p + "mix.left.o", D, H * a["vdim"])
            put(p + "mix.left.q.norm", H * a["dim"], mean=1.0)
            put(p + "mix.left.k.norm", G * a["dim"], mean=1.0)
            put(p + "mix.left.rel", buckets, H, std=1.5)
            R = r["heads"]
            for n, rows in (("q", R * r["dim"]), ("k", R * r["dim"]), ("v", R * r["vdim"]), ("g", R * r["vdim"]), ("i", R), ("f", R)):
                put(f"{p}mix.right.{n}", rows, D)
            put(p + "mix.right.i.b", R, std=1.0, mean=-1.0)
            put(p + "mix.right.f.b", R, std=1.0, mean=3.5)
            put(p + "mix.right.norm", R * r["vdim"], mean=1.0)
            put(p + "mix.right.o", D, R * r["vdim"])
            put(p + "mix.left.out", D, mean=1.0)
            put(p + "mix.right.out", D, mean=1.0)
        put(p + "hc1.in", S, mean=0.6)
        put(p + "hc1.out", S, mean=0.4)
        put(p + "hc1.mix", S, S, std=0.15)
        w[p + "hc1.mix"] = (w[p + "hc1.mix"] + 0.75 * torch.eye(S)).to(torch.bfloat16).float()
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            put(p + "norm2", D, mean=1.0)
            put(p + "mlp.gate", ff, D)
            put(p + "mlp.up", ff, D)
            put(p + "mlp.down", D, ff)
            put(p + "hc2.in", S, mean=0.6)
            put(p + "hc2.out", S, mean=0.4)
            put(p + "hc2.mix", S, S, std=0.15)
            w[p + "hc2.mix"] = (w[p + "hc2.mix"] + 0.75 * torch.eye(S)).to(torch.bfloat16).float()
    return w


def write(path, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()
