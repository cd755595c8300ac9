"""Plain, slow implementation of the Zikezen design for tests: one function per mechanism, one sequence at a time, no code
shared with the package. `cfg` is the dict of a checkpoint's config.json, `w` maps tensor names to tensors."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def layer_runs(cfg):
    """(layer, starts a later pass of the loop) in running order."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    out = [(i, False) for i in range(a)]
    for t in range(lp["times"]):
        out += [(i, t > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


def embedding(cfg, w, toks, first=0):
    return w["embed"][toks] * cfg["embedding"]["scale"] + w["pos"][first:first + len(toks)]


# ------------------------------------------------------------------------------------------------ attention
def frequencies(rot):
    """fp64 angle per position of every pair of dimensions."""
    out, sc = [], rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2 * i / rot["dims"])
        if sc:
            turns = sc["original"] * f / (2 * math.pi)          # over the original context
            if turns < sc["low"]:
                f /= sc["factor"]
            elif turns <= sc["high"]:
                s = (turns - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate(x, positions, rot):
    """x [T, heads, d]: neighbours (0, 1), (2, 3), .. of the first rot.dims dimensions turn together."""
    a = (positions.double()[:, None] * frequencies(rot))[:, None]
    c, s = a.cos().to(x.dtype), a.sin().to(x.dtype)
    out = x.clone()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2] = u * c - v * s
    out[..., 1:rot["dims"]:2] = v * c + u * s
    return out


def queries_keys(w, p, h, m, eps):
    T, at = h.shape[0], torch.arange(h.shape[0])

    def head(n, heads):
        x = (h @ w[p + n].T + w[p + n + ".b"]).view(T, heads, m["dim"])
        return rotate(rms(x, eps) * w[p + n + ".norm"], at, m["rot"])
    return head("q", m["heads"]), head("k", m["kv_heads"])


def visible(i, j, size):
    return 0 <= i - j < size


def sink_softmax(s):
    """Weights e^s / (1 + sum e^s) along the last axis; -inf: not visible."""
    top = s.max(-1, keepdim=True).values.clamp(min=0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attend(q, k, v, m):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H * dv]."""
    T, H, G = q.shape[0], m["heads"], m["kv_heads"]
    i = torch.arange(T)
    gap = i[:, None] - i[None]
    see = (gap >= 0) & (gap < m["mask"]["size"])
    out = torch.zeros(T, H, m["vdim"], dtype=q.dtype)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T * m["scale"]).masked_fill(~see, -math.inf)
        out[:, a] = sink_softmax(s) @ v[:, g]
    return out.reshape(T, -1)


def attention(w, p, h, m, eps):
    q, k = queries_keys(w, p, h, m, eps)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(h.shape[0], m["kv_heads"], m["vdim"])
    return attend(q, k, v, m) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ matrix memory
def decays(z, tau):
    """sigmoid(z)^(1 / tau)"""
    return torch.exp(-(torch.log1p(torch.exp(-z.abs())) + (-z).clamp(min=0)) / tau)


def gla_recurrence(q, k, v, alpha):
    """q, k, alpha [T, H, d], v [T, H, dv] -> [T, H, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out)


def gated_linear_attention(w, p, h, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = ((h @ w[p + n].T).view(T, H, d) for n in "qk")
    v = (h @ w[p + "v"].T).view(T, H, dv)
    alpha = decays((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"], m["tau"]).view(T, H, d)
    o = rms(gla_recurrence(q * d ** -0.5, k, v, alpha), eps) * w[p + "norm"]
    return (o.reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(w, p, h, m, eps):
    return m["left_scale"] * attention(w, p + "left.", h, m["left"], eps) + \
        m["right_scale"] * gated_linear_attention(w, p + "right.", h, m["right"], eps)


# ------------------------------------------------------------------------------------------------ feed-forward
def glu(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, router, correction, top):
    """Weights [T, experts], zero where an expert is not chosen."""
    s = torch.softmax(h @ router.T, -1)
    idx = (s + correction).topk(top, -1).indices
    return torch.zeros_like(s).scatter(1, idx, s.gather(1, idx))


def experts(w, p, h, mlp):
    r = route(h, w[p + "router"], w[p + "correction"], mlp["router"]["top"])
    return sum(r[:, e:e + 1] * glu(w, f"{p}e{e}.", h) for e in range(mlp["router"]["experts"]))


def feed_forward(w, p, h, mlp):
    return glu(w, p, h) if mlp["kind"] == "dense" else experts(w, p, h, mlp)


def token_side(w, p, x, e, eps):
    """The residual's update from the token's own row: x [T, D], e [T, dim]."""
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return rms(y, eps) * w[p + "norm"]


def forward(cfg, weights, tokens, dtype=torch.float64, want_layers=False):
    """Logits [T, vocab] of one sequence (and the residual after every layer run)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, dim = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    toks = torch.as_tensor(tokens)
    norm = lambda x, name: rms(x, eps) * w[name]  # noqa: E731
    x = start = embedding(cfg, w, toks)
    side = w["side.embed"][toks]
    seen = []
    for i, again in layer_runs(cfg):
        p, L = f"l{i}.", cfg["layers"][i]
        if again:
            x = x + start
        x = x + norm(parallel(w, p + "mix.", norm(x, p + "norm1"), L["mixer"], eps), p + "norm1b")
        if L["mlp"] is not None:
            x = x + norm(feed_forward(w, p + "mlp.", norm(x, p + "norm2"), L["mlp"]), p + "norm2b")
        x = x + token_side(w, p + "side.", x, side[:, i * dim:(i + 1) * dim], eps)
        seen.append(x)
    z = norm(x, "final.norm") @ w["head"].T
    cap = cfg["logit_softcap"]
    z = cap * torch.tanh(z / cap)
    return (z, torch.stack(seen)) if want_layers else z
