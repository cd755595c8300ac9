"""Small Roluzen, Tovalix, Zikezen and Zigipel checkpoints with random weights for the layer-stack tests (config.json dict + tensors by name)."""
import json
import os

import torch

from tests import roluzen_oracle, tovalix_oracle, zigipel_oracle, zikezen_oracle


def oracle(cfg):
    return {"Roluzen": roluzen_oracle, "Tovalix": tovalix_oracle, "Zikezen": zikezen_oracle, "Zigipel": zigipel_oracle}[cfg["architecture"]]


# ---- Roluzen

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


# ---- Tovalix
def wkv(heads=3, dim=16, ff=56):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def hgrn2(heads=2, dim=24, vdim=40, ff=72):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def rotary(heads=4, kv_heads=2, dim=16, vdim=24, rot=8, base=900.0, scale=0.6, cap=6.0, chunk=20, kv_from=None, ff=64):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot, "base": base}, "scale": scale,
         "softcap": cap, "mask": {"size": chunk}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def tovalix(layers, width=48, vocab=101, groups=3, side=8, eps=1e-5):
    return {"architecture": "Tovalix", "layers": layers, "norm": {"eps": eps, "groups": groups}, "token_side": {"dim": side},
            "vocab": vocab, "width": width}


# ---- Zikezen
def scaled_rot(dims=8, base=700.0, factor=5.0, low=1.0, high=3.5, original=60):
    return {"dims": dims, "base": base, "scaling": {"factor": factor, "low": low, "high": high, "original": original}}


def sink_attention(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.4, size=20, rot=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
            "rot": rot or scaled_rot()}


def gated(heads=2, dim=24, vdim=40, tau=12.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def beside(left=None, right=None, ff=72, scales=(0.7, 1.3), experts=None):
    """`experts`: (number, chosen), of width ff each."""
    mlp = None if ff is None else {"kind": "dense", "ff": ff}
    if experts:
        mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts[0], "top": experts[1]}}
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left or sink_attention(), "right": right or gated(),
                                                      "left_scale": scales[0], "right_scale": scales[1]}}


def zikezen(layers, width=48, vocab=101, loop=None, side=8, eps=1e-5, cap=12.0, scale=1.7, positions=512):
    return {"architecture": "Zikezen", "embedding": {"scale": scale}, "layers": layers, "logit_softcap": cap,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "max_positions": positions,
            "norm": {"eps": eps}, "token_side": {"dim": side}, "vocab": vocab, "width": width}


# ---- Zigipel
def yarn_rot(dims=8, base=700.0, factor=5.0, fast=3.0, slow=0.5, original=60):
    return {"dims": dims, "base": base, "scaling": {"factor": factor, "fast": fast, "slow": slow, "original": original}}


def distance(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.6, size=20, keep_first=3, ff=56):
    return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                      "mask": {"size": size, "keep_first": keep_first}}}


def latent(heads=3, dim=16, rot_dim=8, vdim=24, rank=40, scale=0.5, size=23, rot=None, ff=40):
    return {"type": "latent_attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale, "mask": {"size": size},
                      "rot": rot or yarn_rot(rot_dim)}}


def zigipel(layers, width=48, vocab=101, loop=None, eps=1e-5, buckets=53, mul_prev=5, mul_cur=3, logit_scale=0.4):
    return {"architecture": "Zigipel", "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "layers": layers, "logit_scale": logit_scale, "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)),
            "norm": {"eps": eps}, "vocab": vocab, "width": width}


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
    # keys and values shared by layers with unequal chunks and query heads
    "shared": tovalix([wkv(), rotary(), hgrn2(ff=None), rotary(heads=2, chunk=33, cap=3.0, kv_from=1, ff=None), wkv(2, 24)]),
    # widths that fit no vector load or tensor-core tile, one norm group, a shared cache read twice
    "uneven": tovalix([hgrn2(3, 12, 6, ff=31), rotary(3, 1, 10, 6, rot=6, chunk=9, cap=40.0, ff=33), wkv(3, 10, ff=45),
                       rotary(3, 1, 10, 6, rot=6, chunk=70, kv_from=1), rotary(3, 1, 10, 6, rot=6, chunk=14, kv_from=1, ff=None)],
                      width=36, vocab=67, groups=1, side=3, eps=1e-3),
    # the head sizes of the tensor-core kernels, values wider than one slice
    "tiles": tovalix([rotary(6, 3, 64, 64, rot=32, chunk=70, scale=0.3, cap=9.0, ff=128), wkv(2, 64, ff=96), hgrn2(2, 104, 136, ff=64),
                      rotary(3, 3, 64, 64, rot=32, chunk=130, scale=0.3, cap=12.0, kv_from=0, ff=None), wkv(1, 128, ff=None)],
                     width=128, vocab=300, groups=4, side=16),
    # a loop over the middle layers, unequal mixers, experts and no feed-forward, the loop's first layer without one before it
    "looped": zikezen([beside(ff=40, experts=(6, 2)), beside(sink_attention(heads=2, kv_heads=2, size=7), gated(3, 16, 24), ff=None,
                                                             scales=(1.1, 0.4)),
                       beside(right=gated(1, 8, 16, tau=1.0), ff=56, experts=(5, 5)), beside()], loop=(0, 3, 3)),
    # widths that fit no vector load or tensor-core tile, one rotated pair, no scaled frequencies, one expert of many
    "ragged": zikezen([beside(sink_attention(3, 1, 10, 6, size=33, rot={"dims": 2, "base": 40.0}), gated(2, 7, 9, tau=5.0), ff=31),
                       beside(sink_attention(3, 3, 6, 14, size=70, rot=scaled_rot(dims=6)), gated(1, 30, 6), ff=13, experts=(9, 1)),
                       beside(ff=None)], width=36, vocab=67, side=3, eps=1e-3, loop=(1, 2, 2), cap=4.0),
    # the sizes of the tensor-core kernels: heads that are stored wider than they are, whole heads, experts
    "blocks": zikezen([beside(sink_attention(6, 3, 40, 56, size=70, scale=0.2, rot=scaled_rot(dims=24)), gated(2, 40, 72), ff=64,
                              experts=(7, 3)),
                       beside(sink_attention(4, 1, 96, 80, size=130, scale=0.15, rot=scaled_rot(dims=96)), gated(1, 104, 136), ff=96),
                       beside(sink_attention(2, 2, 128, 128, size=65, scale=0.1, rot=scaled_rot(dims=64)), gated(3, 64, 64), ff=40,
                              experts=(40, 2))], width=128, vocab=300, side=16, loop=(1, 3, 2)),
    # both mixers with and without feed-forward, small heads on the tensor-core kernels, a loop over the middle
    "pairs": zigipel([distance(), latent(), latent(4, 24, 16, 8, 24, size=70, ff=None), distance(2, 1, 24, 16, size=33, keep_first=40, ff=None)],
                     loop=(1, 3, 2)),
    # widths that fit no vector load or tensor-core tile, the loop from the first layer to the last, kept tokens beyond the window
    "crooked": zigipel([distance(3, 1, 10, 6, size=9, keep_first=12, ff=31), latent(3, 7, 6, 5, 13, size=30, rot=yarn_rot(6, base=40.0), ff=33),
                        latent(1, 12, 2, 9, 50, size=66, ff=None)], width=36, vocab=67, eps=1e-3, loop=(0, 3, 3), buckets=11, mul_prev=1,
                       mul_cur=1, logit_scale=1.0),
    # the sizes of the tensor-core kernels: more heads than one group, wide latents, every pair of head sizes; no loop
    "slabs": zigipel([distance(8, 2, 40, 56, size=70, scale=0.3, keep_first=5, ff=96), latent(20, 96, 64, 128, 136, scale=0.2, size=130, ff=64),
                      distance(4, 4, 128, 112, size=129, scale=0.2, keep_first=1, ff=None), latent(3, 48, 16, 40, 264, scale=0.4, size=65, ff=72),
                      latent(17, 104, 24, 64, 512, scale=0.2, size=200, rot=yarn_rot(24, original=500), ff=None),
                      latent(5, 136, 32, 200, 72, scale=0.2, size=33)], width=128, vocab=300),
}


def weights(cfg, seed=0, buckets=11):
    """Random tensors of the checkpoint, in bf16-representable fp32. Decays reach from fast to very slow, the bias table is
    large and attention is sharp, so that far tokens, window and chunk edges and kept tokens matter."""
    if cfg["architecture"] == "Tovalix":
        return tovalix_weights(cfg, seed)
    if cfg["architecture"] == "Zikezen":
        return zikezen_weights(cfg, seed)
    if cfg["architecture"] == "Zigipel":
        return zigipel_weights(cfg, seed)
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


def tovalix_weights(cfg, seed=0, rank=6):
    g = torch.Generator().manual_seed(seed)
    w = {}

    def put(name, *shape, std=None, mean=0.0, uniform=None):
        x = torch.randn(*shape, generator=g)
        if uniform is not None:
            x = uniform[0] + (uniform[1] - uniform[0]) * torch.rand(*shape, generator=g)
        else:
            x = mean + ((shape[-1] ** -0.5 if len(shape) > 1 else 0.2) if std is None else std) * x
        w[name] = x.to(torch.bfloat16).float()

    D, V, dim, n = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"], len(cfg["layers"])
    put("embed", V, D, std=0.7)
    put("embed.norm", D, mean=1.0)
    put("side.embed", V, n * dim, std=1.0)
    put("head", V, D)
    put("final.norm", D, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        put(p + "norm1", D, mean=1.0)
        if layer["type"] == "wkv":
            C = m["heads"] * m["dim"]
            for s in "rkvgw":
                put(f"{p}mix.mu.{s}", D, uniform=(0.0, 1.0))
            for s in "rkvg":
                put(f"{p}mix.{s}", C, D)
            put(p + "mix.w1", rank, D)
            put(p + "mix.w2", C, rank, std=0.5)
            put(p + "mix.w0", C, uniform=(-7.0, 1.5))
            put(p + "mix.u", m["heads"], m["dim"], std=1.0)
            put(p + "mix.norm", C, mean=1.0)
            put(p + "mix.o", D, C)
        elif layer["type"] == "hgrn2":
            K, C = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for s, rows in (("q", K), ("f", K), ("v", C)):
                put(f"{p}mix.{s}", rows, D)
            put(p + "mix.f.b", K, std=2.0, mean=2.0)
            put(p + "mix.lower", K, uniform=(0.0, 0.99))
            put(p + "mix.norm", m["vdim"], mean=1.0)
            put(p + "mix.o", D, C)
        else:
            H, G = m["heads"], m["kv_heads"]
            own = m.get("kv_from") is None
            for s, rows in (("q", H * m["dim"]),) + ((("k", G * m["dim"]), ("v", G * m["vdim"])) if own else ()):
                put(f"{p}mix.{s}", rows, D)
                put(f"{p}mix.{s}.b", rows, std=0.5)
            put(p + "mix.o", D, H * m["vdim"])
            put(p + "mix.o.b", D)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            put(p + "norm2", D, mean=1.0)
            put(p + "mlp.up", ff, D)
            put(p + "mlp.down", D, ff)
            put(p + "mlp.act", 2, std=1.0)
        put(p + "side.gate", dim, D)
        put(p + "side.proj", D, dim)
        put(p + "side.norm", D, std=0.3)
    return w


ROUTED = 4       # leading dimensions that only the embedding writes and the routers read


def zikezen_weights(cfg, seed=0, rank=8):
    """Routers read a few dimensions that no sublayer writes, and the embedding rows are drawn such that no choice between experts
    is close: rounding then never sends a token to another expert. Which experts a token takes differs from layer to layer."""
    g = torch.Generator().manual_seed(seed)
    w = {}

    def put(name, *shape, std=None, mean=0.0):
        std = (shape[-1] ** -0.5 if len(shape) > 1 else 0.2) if std is None else std
        w[name] = (mean + std * torch.randn(*shape, generator=g)).to(torch.bfloat16).float()

    D, V, dim, n = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"], len(cfg["layers"])
    if D % 8:
        rank = 5
    put("embed", V, D, std=0.5)
    put("pos", cfg["max_positions"], D, std=0.4)
    put("side.embed", V, n * dim, std=1.0)
    put("head", V, D, std=3.0 * D ** -0.5)
    put("final.norm", D, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, a, r, mlp = f"l{i}.", layer["mixer"]["left"], layer["mixer"]["right"], layer["mlp"]
        for s in ("norm1",) + (() if mlp is None else ("norm2",)):
            put(p + s, D, mean=1.0)
        for s in ("norm1b",) + (() if mlp is None else ("norm2b",)):
            put(p + s, D, mean=0.6)
            w[p + s][:ROUTED] = 0
        H, G = a["heads"], a["kv_heads"]
        for s, rows in (("q", H * a["dim"]), ("k", G * a["dim"]), ("v", G * a["vdim"])):
            put(f"{p}mix.left.{s}", rows, D)
            put(f"{p}mix.left.{s}.b", rows, std=0.5)
        put(p + "mix.left.q.norm", a["dim"], mean=1.3, std=0.5)
        put(p + "mix.left.k.norm", a["dim"], mean=1.3, std=0.5)
        put(p + "mix.left.o", D, H * a["vdim"])
        K, C = r["heads"] * r["dim"], r["heads"] * r["vdim"]
        for s, rows in (("q", K), ("k", K), ("v", C), ("g", C)):
            put(f"{p}mix.right.{s}", rows, D)
        put(p + "mix.right.a1", rank, D)
        put(p + "mix.right.a2", K, rank, std=0.7)
        put(p + "mix.right.a2.b", K, std=3.0)
        put(p + "mix.right.norm", r["vdim"], mean=1.0)
        put(p + "mix.right.o", D, C)
        if mlp is not None and mlp["kind"] == "dense":
            for s, shape in (("gate", (mlp["ff"], D)), ("up", (mlp["ff"], D)), ("down", (D, mlp["ff"]))):
                put(f"{p}mlp.{s}", *shape)
        elif mlp is not None:
            F, E = mlp["expert"]["ff"], mlp["router"]["experts"]
            for e in range(E):
                for s, shape in (("gate", (F, D)), ("up", (F, D)), ("down", (D, F))):
                    put(f"{p}mlp.e{e}.{s}", *shape)
            put(p + "mlp.router", E, D, std=1.3)
            w[p + "mlp.router"][:, ROUTED:] = 0
            put(p + "mlp.correction", E, std=0.2, mean=0.5)
            w[p + "norm2"][:ROUTED] = 1
        put(p + "side.gate", dim, D)
        put(p + "side.proj", D, dim)
        put(p + "side.norm", D, std=0.3)
        w[p + "side.norm"][:ROUTED] = 0
    w["pos"][:, :ROUTED] = 0
    kept = []
    while sum(map(len, kept)) < V:
        rows = (2 * torch.randn(20 * V, ROUTED, generator=g)).to(torch.bfloat16).float()
        clear = torch.ones(len(rows), dtype=torch.bool)
        for i, layer in enumerate(cfg["layers"]):
            if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe" and layer["mlp"]["router"]["top"] < layer["mlp"]["router"]["experts"]:
                top = layer["mlp"]["router"]["top"]
                for size in torch.linspace(0.1, 1.4, 150):             # whatever the norm makes of a row's size
                    s = torch.softmax(size * rows @ w[f"l{i}.mlp.router"][:, :ROUTED].T, -1) + w[f"l{i}.mlp.correction"]
                    s = s.topk(top + 1, -1).values
                    clear &= s[:, top - 1] - s[:, top] > 0.015
        kept.append(rows[clear])
    w["embed"][:, :ROUTED] = torch.cat(kept)[:V] / cfg["embedding"]["scale"]
    w["embed"] = w["embed"].to(torch.bfloat16).float()
    return w


def zigipel_weights(cfg, seed=0):
    """Attention is sharp, the distance takes a few units off a far key's score, and sinks stand among the scores."""
    g = torch.Generator().manual_seed(seed)
    w = {}

    def put(name, *shape, std=None, mean=0.0, uniform=None):
        x = torch.randn(*shape, generator=g)
        if uniform is not None:
            x = uniform[0] + (uniform[1] - uniform[0]) * torch.rand(*shape, generator=g)
        else:
            x = mean + ((shape[-1] ** -0.5 if len(shape) > 1 else 0.2) if std is None else std) * x
        w[name] = x.to(torch.bfloat16).float()

    D, V = cfg["width"], cfg["vocab"]
    put("embed", V, D, std=0.7)
    put("bigram", cfg["embedding"]["bigram"]["buckets"] + 1, D, std=0.7)
    if cfg["loop"]:
        put("loop.in", D, 2 * D)
        put("loop.step", cfg["loop"]["times"], D, std=0.5)
    put("head", V, D, std=3.0 * D ** -0.5)
    put("final.norm", D, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m, H = f"l{i}.", layer["mixer"], layer["mixer"]["heads"]
        put(p + "norm1", D, mean=1.0)
        put(p + "shift", D, uniform=(0.0, 1.0))
        if layer["type"] == "attention":
            G = m["kv_heads"]
            for s, rows in (("q", H * m["dim"]), ("k", G * m["dim"]), ("v", G * m["vdim"]), ("g", H)):
                put(f"{p}mix.{s}", rows, D)
            put(p + "mix.r1", H, uniform=(0.1, 0.8))
            put(p + "mix.r2", H, uniform=(0.1, 2.0))
        else:
            R = m["kv_rank"]
            put(p + "mix.q", H * (m["dim"] + m["rot_dim"]), D)
            put(p + "mix.dkv", R + m["rot_dim"], D)
            put(p + "mix.dkv.norm", R, mean=1.0)
            put(p + "mix.uk", H * m["dim"], R)
            put(p + "mix.uv", H * m["vdim"], R)
        put(p + "mix.sink", H, std=1.5, mean=1.0)
        put(p + "mix.o", D, H * m["vdim"])
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            for s, shape in (("gate", (ff, D)), ("up", (ff, D)), ("down", (D, ff))):
                put(f"{p}mlp.{s}", *shape)
                put(f"{p}mlp.{s}.b", shape[0], std=0.5)
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
