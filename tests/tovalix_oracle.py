"""Plain, slow implementation of the Tovalix design for tests: one function per mechanism, one sequence at a time, no code
shared with the package. `cfg` is the dict of a checkpoint's config.json, `w` maps tensor names to tensors."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, weight, groups, eps):
    """RMS norm of `groups` equal consecutive parts of the last axis, then one weight over the whole of it."""
    parts = x.reshape(*x.shape[:-1], groups, -1)
    return rms(parts, eps).reshape(x.shape) * weight


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def xielu(z, p, q):
    neg = (0.5 + softplus(q)) * (torch.exp(z.clamp(max=0)) - 1 - z) + z / 2
    return torch.where(z > 0, softplus(p) * z * z + z / 2, neg)


def mlp(w, p, h):
    return xielu(h @ w[p + "up"].T, w[p + "act"][0], w[p + "act"][1]) @ w[p + "down"].T


def token_side(w, p, x, e, eps):
    """The residual's update from the token's own row: x [T, D], e [T, dim]."""
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return rms(y, eps) * w[p + "norm"]


def token_shift(h, mu):
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def wkv_recurrence(r, k, v, decay, u):
    """r, k, decay [T, H, d], v [T, H, dv], u [H, d] -> [T, H, dv]."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[2], dtype=r.dtype)
    out = []
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t]))
        S = decay[t][:, :, None] * S + kv
    return torch.stack(out)


def wkv(w, p, h, m, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    mix = {n: token_shift(h, w[p + "mu." + n]) for n in "rkvgw"}
    r, k, v = (torch.reshape(mix[n] @ w[p + n].T, (T, H, d)) for n in "rkv")
    gate = silu(mix["g"] @ w[p + "g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).view(T, H, d)
    o = wkv_recurrence(r, k, v, decay, w[p + "u"])
    return (rms(o, eps).reshape(T, H * d) * w[p + "norm"] * gate) @ w[p + "o"].T


def hgrn2_recurrence(q, f, v):
    """q, f [T, H, d], v [T, H, dv] -> [T, H, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out)


def hgrn2(w, p, h, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).view(T, H, d)
    low = w[p + "lower"]
    f = (low + (1 - low) * torch.sigmoid(h @ w[p + "f"].T + w[p + "f.b"])).view(T, H, d)
    o = hgrn2_recurrence(q, f, (h @ w[p + "v"].T).view(T, H, dv))
    return (rms(o, eps) * w[p + "norm"]).reshape(T, H * dv) @ w[p + "o"].T


def rotate(x, positions, dims, base):
    """x [T, heads, d]: the first `dims` of each head turn, element i together with element i + dims / 2."""
    half = dims // 2
    freq = torch.tensor([base ** (-2 * i / dims) for i in range(half)], dtype=torch.float64)
    a = (positions.double()[:, None] * freq)[:, None].to(x.dtype)
    a, b, rest = (a.cos(), a.sin()), (x[..., :half], x[..., half:dims]), x[..., dims:]
    return torch.cat([b[0] * a[0] - b[1] * a[1], b[1] * a[0] + b[0] * a[1], rest], -1)


def visible(i, j, chunk):
    return j <= i and i // chunk == j // chunk


def keys_values(w, p, h, m, eps):
    T, G = h.shape[0], m["kv_heads"]
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, m["dim"])
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, m["vdim"])
    return rms(rotate(k, torch.arange(T), m["rot"]["dims"], m["rot"]["base"]), eps), v


def attention(w, p, h, m, eps, kv):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, m["dim"])
    q = rms(rotate(q, torch.arange(T), m["rot"]["dims"], m["rot"]["base"]), eps)
    k, v = kv
    cap, size = m["softcap"], m["mask"]["size"]
    i = torch.arange(T)
    see = (i[None] <= i[:, None]) & (i[None] // size == i[:, None] // size)
    out = torch.zeros(T, H, m["vdim"], dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        s = cap * torch.tanh(q[:, a] @ k[:, g].T * m["scale"] / cap)
        out[:, a] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, g]
    return out.reshape(T, -1) @ w[p + "o"].T + w[p + "o.b"]


def forward(cfg, weights, tokens, dtype=torch.float64, want_layers=False):
    """Logits [T, vocab] of one sequence (and the residual after every layer)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, groups, dim = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["token_side"]["dim"]
    toks = torch.as_tensor(tokens)
    norm = lambda x, name: group_norm(x, w[name], groups, eps)  # noqa: E731
    x = norm(w["embed"][toks], "embed.norm")
    side = w["side.embed"][toks]
    kv, seen = {}, []
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = norm(x, p + "norm1")
        if L["type"] == "wkv":
            y = wkv(w, p + "mix.", h, m, eps)
        elif L["type"] == "hgrn2":
            y = hgrn2(w, p + "mix.", h, m, eps)
        else:
            j = m.get("kv_from")
            if j is None:
                kv[i] = keys_values(w, p + "mix.", h, m, eps)
            y = attention(w, p + "mix.", h, m, eps, kv[i if j is None else j])
        x = x + y
        if L["mlp"] is not None:
            x = x + mlp(w, p + "mlp.", norm(x, p + "norm2"))
        x = x + token_side(w, p + "side.", x, side[:, i * dim:(i + 1) * dim], eps)
        seen.append(x)
    z = norm(x, "final.norm") @ w["head"].T
    return (z, torch.stack(seen)) if want_layers else z
