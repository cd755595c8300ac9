"""Plain, slow implementation of the Zigipel design for tests: one function per mechanism, one sequence at a time, no code
shared with the package. `cfg` is the dict of a checkpoint's config.json, `w` maps tensor names to tensors."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def layer_runs(cfg):
    """(layer, pass of the loop that it begins or None) in running order."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    out = [(i, None) for i in range(a)]
    for t in range(lp["times"]):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


# ------------------------------------------------------------------------------------------------ embedding
def bigram_rows(toks, b):
    """Row of the pair table per token; the row behind the buckets for a sequence's first token."""
    toks = [int(t) for t in toks]
    return [b["buckets"]] + [(toks[i - 1] * b["mul_prev"] + toks[i] * b["mul_cur"]) % b["buckets"] for i in range(1, len(toks))]


def embedding(cfg, w, toks):
    return w["embed"][toks] + w["bigram"][bigram_rows(toks, cfg["embedding"]["bigram"])]


def loop_input(w, x, start, t):
    return torch.cat([x, start], -1) @ w["loop.in"].T + w["loop.step"][t]


# ------------------------------------------------------------------------------------------------ attention
def token_shift(h, mu):
    """h [T, D] -> h + (row before - h) * mu; zeros before the first token."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def visible(i, j, mask):
    return j <= i and (i - j < mask["size"] or j < mask.get("keep_first", 0))


def seen(T, mask):
    i = torch.arange(T)
    gap = i[:, None] - i[None]
    return (gap >= 0) & ((gap < mask["size"]) | (i[None] < mask.get("keep_first", 0)))


def distance_bias(gap, r1, r2):
    return r1 * torch.log1p(r2 * gap)


def sink_softmax(s, sink):
    """Weights e^s / (e^sink + sum e^s) along the last axis; -inf: not visible."""
    top = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (torch.exp(sink - top) + e.sum(-1, keepdim=True))


def attend(q, k, v, m, r1, r2, sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; r1, r2, sink [H] -> [T, H, dv]."""
    T, H, G = q.shape[0], m["heads"], m["kv_heads"]
    i = torch.arange(T)
    gap = (i[:, None] - i[None]).clamp(min=0).to(q.dtype)
    out = []
    for a in range(H):
        g = a // (H // G)
        s = q[:, a] @ k[:, g].T * m["scale"] - distance_bias(gap, r1[a], r2[a])
        out.append(sink_softmax(s.masked_fill(~seen(T, m["mask"]), -math.inf), sink[a]) @ v[:, g])
    return torch.stack(out, 1)


def attention(w, p, h, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w[p + "q"].T).view(T, H, m["dim"])
    k = (h @ w[p + "k"].T).view(T, G, m["dim"])
    v = rms((h @ w[p + "v"].T).view(T, G, m["vdim"]), eps)
    o = attend(q, k, v, m, w[p + "r1"], w[p + "r2"], w[p + "sink"])
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ latent attention
def frequencies(rot):
    """fp64 angle per position of every pair of dimensions."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2 * i / n) for i in range(n // 2)]
    if sc:
        def dim(turns):
            return n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(dim(sc["fast"])), 0), min(math.ceil(dim(sc["slow"])), n - 1)
        for i in range(n // 2):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f[i] = f[i] / sc["factor"] * ramp + f[i] * (1 - ramp)
    return torch.tensor(f, dtype=torch.float64)


def rotate(x, positions, rot):
    """x [T, .., d]: dimension i of the first rot.dims turns with i + dims / 2."""
    n = rot["dims"]
    a = positions.double()[:, None] * frequencies(rot)
    a = a.view(len(positions), *[1] * (x.dim() - 2), n // 2)
    size = 0.1 * math.log(rot["scaling"]["factor"]) + 1 if rot.get("scaling") else 1.0
    c, s = (size * a.cos()).to(x.dtype), (size * a.sin()).to(x.dtype)
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


def latents(w, p, h, m, eps):
    """(normed latent [T, rank], rotated key part [T, rot_dim])."""
    z = h @ w[p + "dkv"].T
    return rms(z[:, :m["kv_rank"]], eps) * w[p + "dkv.norm"], rotate(z[:, m["kv_rank"]:], torch.arange(h.shape[0]), m["rot"])


def latent_attend(q, qr, k, kr, v, m, sink):
    """q, k [T, H, d], v [T, H, dv], rotated parts qr [T, H, r], kr [T, r] -> [T, H, dv]."""
    see, out = seen(q.shape[0], m["mask"]), []
    for a in range(m["heads"]):
        s = (q[:, a] @ k[:, a].T + qr[:, a] @ kr.T) * m["scale"]
        out.append(sink_softmax(s.masked_fill(~see, -math.inf), sink[a]) @ v[:, a])
    return torch.stack(out, 1)


def latent_attention(w, p, h, m, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    q = (h @ w[p + "q"].T).view(T, H, d + m["rot_dim"])
    c, kr = latents(w, p, h, m, eps)
    k, v = (c @ w[p + "uk"].T).view(T, H, d), (c @ w[p + "uv"].T).view(T, H, m["vdim"])
    o = latent_attend(q[..., :d], rotate(q[..., d:], torch.arange(T), m["rot"]), k, kr, v, m, w[p + "sink"])
    return o.reshape(T, -1) @ w[p + "o"].T


MIXERS = {"attention": attention, "latent_attention": latent_attention}


# ------------------------------------------------------------------------------------------------ feed-forward, model
def feed_forward(w, p, h):
    lin = lambda x, n: x @ w[p + n].T + w[p + n + ".b"]  # noqa: E731
    return lin(gelu_tanh(lin(h, "gate")) * lin(h, "up"), "down")


def forward(cfg, weights, tokens, dtype=torch.float64, want_layers=False):
    """Logits [T, vocab] of one sequence (and the residual after every layer run)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, toks = cfg["norm"]["eps"], torch.as_tensor(tokens)
    x = start = embedding(cfg, w, toks)
    after = []
    for i, t in layer_runs(cfg):
        p, L = f"l{i}.", cfg["layers"][i]
        if t is not None:
            x = loop_input(w, x, start, t)
        h = rms(x, eps) * w[p + "norm1"]
        y = MIXERS[L["type"]](w, p + "mix.", token_shift(h, w[p + "shift"]), L["mixer"], eps)
        if L["mlp"] is not None:
            y = y + feed_forward(w, p + "mlp.", h)
        x = x + y
        after.append(x)
    z = rms(x, eps) * w["final.norm"] @ w["head"].T * cfg["logit_scale"]
    return (z, torch.stack(after)) if want_layers else z
