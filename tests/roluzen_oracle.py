"""Plain, slow implementation of the Roluzen design for tests: one function per mechanism, one sequence at a time, no
code shared with the package. `cfg` is the dict of a checkpoint's config.json, `w` maps tensor names to tensors."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def dense_mlp(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def distance_bucket(n, rows, far):
    """Bucket of distance n: one per distance in the lower half, logarithmic up to `far` in the upper half."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def visible(i, j, size, keep_first):
    return j <= i and (i - j < size or j < keep_first)


def biased_window_attention(w, p, h, m, eps):
    """Full sequence h [T, D] -> [T, D]: whole-projection query / key norm, learned distance bias, sliding window with
    kept first tokens, softmax, output gate."""
    T = h.shape[0]
    H, G, dq, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(T, H, dq)
    k = (rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(T, G, dq)
    v = (h @ w[p + "v"].T).view(T, G, dv)
    rel = w[p + "rel"]
    size, keep = m["mask"]["size"], m["mask"]["keep_first"]
    bucket = torch.tensor([distance_bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)])
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    see = (j <= i) & ((i - j < size) | (j < keep))
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        s = q[:, a] @ k[:, g].T * m["scale"] + rel[bucket[(i - j).clamp(min=0)], a]
        out[:, a] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, g]
    return (out.reshape(T, H * dv) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def matrix_memory(w, p, h, m, eps):
    """mLSTM over the full sequence, token by token."""
    T = h.shape[0]
    H, dk, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).view(T, H, dk) * dk ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, dk)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    ig = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    fg = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    S = torch.zeros(H, dk, dv, dtype=h.dtype)
    n = torch.zeros(H, dk, dtype=h.dtype)
    mx = torch.zeros(H, dtype=h.dtype)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        new = torch.maximum(fg[t] + mx, ig[t])
        a, b = torch.exp(fg[t] + mx - new), torch.exp(ig[t] - new)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        mx = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-mx)) + 1e-6
        out[t] = torch.einsum("hkv,hk->hv", S, q[t]) / den[:, None]
    y = rms(out, eps).reshape(T, H * dv) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


def parallel_mixer(w, p, h, m, eps):
    a = biased_window_attention(w, p + "left.", h, m["left"], eps)
    b = matrix_memory(w, p + "right.", h, m["right"], eps)
    return 0.5 * (rms(a, eps) * w[p + "left.out"] + rms(b, eps) * w[p + "right.out"])


def causal_conv(u, taps, bias):
    """u [T, C], taps [C, K]: the last column weighs the current token."""
    K = taps.shape[1]
    pad = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u])
    return sum(pad[j:j + u.shape[0]] * taps[:, j] for j in range(K)) + bias


def rglru_mixer(w, p, h, m):
    T = h.shape[0]
    nb = m["blocks"]
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    ub = u.view(T, nb, -1)
    r = torch.sigmoid(torch.einsum("boi,tbi->tbo", w[p + "ra"], ub) + w[p + "ra.b"]).reshape(T, -1)
    i = torch.sigmoid(torch.einsum("boi,tbi->tbo", w[p + "ri"], ub) + w[p + "ri.b"]).reshape(T, -1)
    loga = -8.0 * r * torch.nn.functional.softplus(w[p + "lam"])
    a = torch.exp(loga)
    s = torch.zeros(u.shape[1], dtype=u.dtype)
    out = torch.zeros_like(u)
    for t in range(T):
        s = a[t] * s + torch.sqrt(1 - a[t] ** 2) * i[t] * u[t]
        out[t] = s
    return (out * y) @ w[p + "o"].T


def layer_runs(cfg):
    """Layer index of every pass, the looped range unrolled."""
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return list(range(n))
    a, b = lp["start"], lp["stop"]
    return list(range(a)) + list(range(a, b)) * lp["times"] + list(range(b, n))


def hyper_in(w, p, x):
    return torch.einsum("s,tsd->td", w[p + "in"], x)


def hyper_out(w, p, x, y):
    return torch.einsum("st,nsd->ntd", w[p + "mix"], x) + w[p + "out"][None, :, None] * y[:, None, :]


def forward(cfg, weights, tokens, dtype=torch.float64, want_layers=False):
    """Logits [T, vocab] of one sequence (and, per layer run, the sum of the streams)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)][:, None, :].repeat(1, cfg["streams"], 1)
    seen = []
    for i in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        h = rms(hyper_in(w, p + "hc1.", x), eps) * w[p + "norm1"]
        y = rglru_mixer(w, p + "mix.", h, L["mixer"]) if L["type"] == "rglru" else \
            parallel_mixer(w, p + "mix.", h, L["mixer"], eps)
        x = hyper_out(w, p + "hc1.", x, y)
        if L["mlp"] is not None:
            h = rms(hyper_in(w, p + "hc2.", x), eps) * w[p + "norm2"]
            x = hyper_out(w, p + "hc2.", x, dense_mlp(w, p + "mlp.", h))
        seen.append(x.sum(1))
    z = (rms(x.sum(1), eps) * w["final.norm"]) @ w["head"].T
    return (z, torch.stack(seen)) if want_layers else z
